// What the recurrences with a matrix per head share: asynchronous copies, sums over lanes, the convolution in front of the delta
// rules, arithmetic on pairs.
#pragma once
#include "common.cuh"
#include <cstdlib>

namespace memory {


constexpr int STAGES = 3;          // one at hand, two on their way
constexpr int GROUP = 4;           // tokens taken together (a stage's tokens are a multiple)
constexpr int MAX_TAPS = 16;

__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ void copy4_async(float* dst_smem, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst_smem)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy16_async(float* dst_smem, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst_smem)), "l"(src) : "memory");
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copies_wait_all_but_one() { asm volatile("cp.async.wait_group 1;" ::: "memory"); }

// N sums over groups of L lanes at once: at every step a lane keeps one half of its values and hands the other over, so that
// N values cost about N exchanges, not N log L.  Afterwards value i is in v[i % max(1, N / L)] of lane i / max(1, N / L) of the
// group, times L / N where the group has more lanes than values (the lanes in between hold copies).
template <int N, int L>
__device__ __forceinline__ void scatter_sum(float* v, int lane) {
    if constexpr (L > 1) {
        constexpr int x = L / 2;
        if constexpr (N > 1) {
            const bool up = (lane & x) != 0;
#pragma unroll
            for (int n = 0; n < N / 2; ++n) {
                const float keep = up ? v[n + N / 2] : v[n], give = up ? v[n] : v[n + N / 2];
                v[n] = keep + __shfl_xor_sync(0xffffffffu, give, x);
            }
            scatter_sum<N / 2, x>(v, lane);
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], x);
            scatter_sum<1, x>(v, lane);
        }
    }
}
template <int N, int L> struct Scattered {
    static constexpr int per_lane = N / L > 1 ? N / L : 1, stride = L / N > 1 ? L / N : 1;
};

// ---- prepare -----------------------------------------------------------------------------------------------------------
struct PrepareArgs {
    const float* proj;       // [T, >= x_off + CH]; CH = 2 G K + H V channels [q | k | v]
    long long proj_stride;
    const float* conv_w;     // [taps, CH]
    float* state;            // + slot * stride: [taps - 1, CH]
    long long state_stride;
    const int* tok_entry;
    const int* entry_q_start;
    const int* entry_slot;
    float* u;                // [T, CH]
    float* table;            // [H, T, 12]: decay g, beta, two unused; k . q; for j = 1, 2, 3 tokens back in the group (0 beyond it)
                             // k_back . k and k_back . q; one unused
    const float* a_log;
    const float* dt_bias;
    int decay_off, step_off; // columns of the raw decays and steps in proj, one per head
    int x_off, taps, n_tokens, G, H, K, V, CH, move_tail;
};

// convolution and silu of channels c .. c + VEC of token t; with move_tail (a step of single tokens) the thread that owns
// the channels also moves the tail on
template <int VEC>
__device__ __forceinline__ void conv_silu(const PrepareArgs& a, int t, int first, float* tail, int c, float* v) {
    float acc[VEC], x[VEC], w[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) acc[k] = 0.f;
    for (int j = 0; j < a.taps; ++j) {
        const int src = t - first - (a.taps - 1 - j);
        const float* p = src >= 0 ? a.proj + (size_t)(first + src) * a.proj_stride + a.x_off + c
                                  : tail + (size_t)(a.taps - 1 + src) * a.CH + c;
        const float* q = a.conv_w + (size_t)j * a.CH + c;
        if constexpr (VEC == 4) {
            const float4 f = *reinterpret_cast<const float4*>(p), g = *reinterpret_cast<const float4*>(q);
            x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
            w[0] = g.x; w[1] = g.y; w[2] = g.z; w[3] = g.w;
        } else {
            x[0] = p[0];
            w[0] = q[0];
        }
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            acc[k] = fmaf(w[k], x[k], acc[k]);
            if (a.move_tail && j > 0) tail[(size_t)(j - 1) * a.CH + c + k] = x[k];
        }
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = silu_f(acc[k]);
}

constexpr int DELTA_ROW = 12, GATED_ROW = 4;         // floats a token and head has in the scan's table

template <int VEC> __device__ __forceinline__ void put(float* p, const float* v) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else p[0] = v[0];
}

constexpr int PREP_WARPS = 8;
constexpr int MAX_K = 512;

struct Window { float w[4][4], x[3][4]; };
__device__ __forceinline__ void load4f(const float* p, float* v) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void window_weights(Window& win, const PrepareArgs& a, int c) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        win.w[j][0] = win.w[j][1] = win.w[j][2] = win.w[j][3] = 0.f;
        if (j >= 4 - a.taps) load4f(a.conv_w + (size_t)(j - (4 - a.taps)) * a.CH + c, win.w[j]);
    }
}
__device__ __forceinline__ void window_start(Window& win, const PrepareArgs& a, int t, int first, const float* tail, int c) {
#pragma unroll
    for (int j = 0; j < 3; ++j) {
        const int src = t - first - (3 - j);
        win.x[j][0] = win.x[j][1] = win.x[j][2] = win.x[j][3] = 0.f;
        if (src >= 0) load4f(a.proj + (size_t)(first + src) * a.proj_stride + a.x_off + c, win.x[j]);
        else if (a.taps - 1 + src >= 0) load4f(tail + (size_t)(a.taps - 1 + src) * a.CH + c, win.x[j]);
    }
}
// the convolution at the next token, whose input is x; the window moves on
__device__ __forceinline__ void window_next(Window& win, const float* x, float* v) {
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        float acc = win.w[0][k] * win.x[0][k];
        acc = fmaf(win.w[1][k], win.x[1][k], acc);
        acc = fmaf(win.w[2][k], win.x[2][k], acc);
        acc = fmaf(win.w[3][k], x[k], acc);
        win.x[0][k] = win.x[1][k], win.x[1][k] = win.x[2][k], win.x[2][k] = x[k];
        v[k] = silu_f(acc);
    }
}

// Two 32-bit numbers in one register pair, and the arithmetic that works on both at once.
typedef unsigned long long f2;
__device__ __forceinline__ f2 f2_of(float a, float b) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float f2_sum(f2 v) {
    float a, b;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
    return a + b;
}
__device__ __forceinline__ f2 f2_fma(f2 a, f2 b, f2 c) {
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 f2_mul(f2 a, f2 b) {
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ f2 f2_add(f2 a, f2 b) {
    f2 r;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

}  // namespace memory
