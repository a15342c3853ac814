// What the recurrences with a matrix per head share (outer_memory.cu says what they are): the convolution in front of the delta
// rules, and the scan with its launch.  The rules are instantiated in files of their own, which compile side by side.
#pragma once
#include "common.cuh"
#include <cstdlib>

namespace memory {


constexpr int STAGES = 3;          // one at hand, two on their way
constexpr int GROUP = 4;           // tokens taken together (a stage's tokens are a multiple)
constexpr int MAX_TAPS = 16;
enum : int { RULE_DELTA = 0, RULE_GATED = 1, RULE_CHANNEL = 2, RULE_DECAYED = 3 };

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

// ---- scan --------------------------------------------------------------------------------------------------------------
struct ScanArgs {
    const float* src;        // rows of q, k and v: [T, >= ...]
    const float* table;      // [H, n_tokens, 12 or 4]: a token's gates (delta: see PrepareArgs; gated: what S is multiplied by,
                             // what k v^T is multiplied by, exp(-m), one unused)
    const float* gates;      // gated, steps of single tokens: rows of the raw gates instead, worked out here
    float* state;            // + slot * stride + s_off: S [H, W, K], then (gated) m [H, W]
    const int* entry_q_start;
    const int* entry_q_len;
    const int* entry_slot;
    float* y;                // [T, H * V]
    float* den;              // gated: [T, H], what o is divided by
    long long src_stride, gate_stride, state_stride, s_off;
    // channel, decayed: one more vector per token and head, [T, H K] (what a token is written with; its decays); channel: the
    // decays of a whole group, in the row of its last token
    const float* aux;
    const float* group_decay;
    long long aux_stride;
    int q_off, k_off, v_off, in_off, forget_off, n_tokens;
    int H, G, K, V, W, wide;
    float q_scale, cap;
};

__device__ __forceinline__ float log_input(float raw, float cap) { return cap * tanhf(raw / cap); }
__device__ __forceinline__ float log_forget(float raw, float cap) { return -softplus_f(-cap * tanhf(raw / cap)); }

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

// Rows of 16-byte chunks into shared memory, the warp's lanes over the chunks of one row after the other.
struct Lanes { int tok, ch, d_tok, d_ch; };          // a lane's first row and chunk, and how far 32 chunks on lies
__device__ __forceinline__ Lanes lanes_over(int chunks, int lane) { return {lane / chunks, lane % chunks, 32 / chunks, 32 % chunks}; }
__device__ __forceinline__ void copy_rows(float* dst, int dst_stride, const float* src, long long src_stride, int chunks, int rows, Lanes at) {
    float* d = dst + at.tok * dst_stride + at.ch * 4;
    const float* p = src + at.tok * src_stride + at.ch * 4;
    const int d_step = at.d_tok * dst_stride + at.d_ch * 4, d_wrap = dst_stride - chunks * 4;
    const long long p_step = at.d_tok * src_stride + at.d_ch * 4, p_wrap = src_stride - chunks * 4;
    int tok = at.tok, ch = at.ch;
#pragma unroll 4
    while (tok < rows) {
        copy16_async(d, p);
        d += d_step, p += p_step, tok += at.d_tok, ch += at.d_ch;
        if (ch >= chunks) ch -= chunks, ++tok, d += d_wrap, p += p_wrap;
    }
}

// The last warp of a block brings the tokens in and writes the results of the stage before; the
// others only walk through the stage at hand.  One barrier a stage.
// A thread holds its rows of CPT neighbouring columns, so that what it reads of a token serves all of them.
template <int RULE> struct ScanPlan {
    static constexpr bool delta = RULE == RULE_DELTA || RULE == RULE_CHANNEL;            // the rule reads before it writes
    static constexpr bool aux = RULE == RULE_CHANNEL || RULE == RULE_DECAYED;
    static constexpr int row = delta ? DELTA_ROW : RULE == RULE_GATED ? GATED_ROW : 0;   // floats of a token's gates
    static constexpr int tch = aux ? 8 : 16;                                             // tokens a stage holds
    static constexpr int group_rows = RULE == RULE_CHANNEL ? tch / GROUP : 0;            // rows of group decays
    static size_t smem_floats(int Kp, int cols) {
        return (size_t)STAGES * (tch * ((aux ? 3 : 2) * Kp + row + cols) + group_rows * Kp) + 2 * tch * cols;
    }
};

template <int RULE, int NR, int LG, int C, int CPT>
__global__ void __launch_bounds__(288) memory_scan_kernel(const ScanArgs a) {
    using Plan = ScanPlan<RULE>;
    constexpr int TCH = Plan::tch, Kp = NR * LG, NP = NR / 2, ROW = Plan::row, GROWS = Plan::group_rows;
    constexpr bool RAW_GATES = RULE == RULE_GATED && C == 1, AUX = Plan::aux;
    extern __shared__ __align__(16) float sm[];
    const int nc = blockDim.x - 32;                  // threads that hold columns
    const int COLS = nc / LG * CPT;
    float* ks = sm;                                  // [STAGES][TCH][Kp]
    float* qs = ks + STAGES * TCH * Kp;              // [STAGES][TCH][Kp]
    float* xs = qs + STAGES * TCH * Kp;              // [STAGES][TCH][Kp] (AUX)
    float* gs = xs + (AUX ? STAGES * TCH * Kp : 0);  // [STAGES][GROWS][Kp] a group's decays (channel)
    float* ts = gs + STAGES * GROWS * Kp;            // [STAGES][TCH][ROW] the tokens' gates
    float* vs = ts + STAGES * TCH * ROW;             // [STAGES][TCH][COLS]
    float* ys = vs + STAGES * TCH * COLS;            // [2][TCH][COLS]
    __shared__ float m_end;
    pdl_launch_dependents();
    const int e = blockIdx.x, h = blockIdx.y, pb = blockIdx.z;
    const int n_new = a.entry_q_len[e];
    if (n_new <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31;
    const bool producer = tid >= nc;
    const int first = a.entry_q_start[e];
    const int kvh = h / (a.H / a.G);
    float* S_head = a.state + (long long)a.entry_slot[e] * a.state_stride + a.s_off + (size_t)h * a.W * a.K;
    float* m_head = a.state + (long long)a.entry_slot[e] * a.state_stride + a.s_off + (size_t)a.H * a.W * a.K + (size_t)h * a.W;
    const int n_stages = (n_new + TCH - 1) / TCH;
    // columns of k and q beyond K are zero in all stages, for good
    for (int i = tid; i < STAGES * TCH * (Kp - a.K); i += blockDim.x) {
        const int tt = i / (Kp - a.K), n = a.K + i % (Kp - a.K);
        ks[tt * Kp + n] = 0.f;
        qs[tt * Kp + n] = 0.f;
        if (AUX) xs[tt * Kp + n] = 0.f;
        if (tt < STAGES * GROWS) gs[tt * Kp + n] = 0.f;
    }
    if (producer) {
        pdl_wait();
        // q, k, v and gates of a stage's tokens, in chunks of 16 bytes where rows start on such boundaries
        const int v_cols = max(0, min(COLS, a.V - pb * COLS));        // columns of v here (the gated rule's ones lie behind them)
        const Lanes over_k = lanes_over(max(1, a.K / 4), lane), over_v = lanes_over(max(1, v_cols / 4), lane);
        auto copy = [&](int s) {
            const int c0 = s * TCH, nt = min(TCH, n_new - c0), buf = s % STAGES;
            const float* row = a.src + (size_t)(first + c0) * a.src_stride;
            const float* qr = row + a.q_off + (size_t)kvh * a.K;
            const float* kr = row + a.k_off + (size_t)kvh * a.K;
            const float* vr = row + a.v_off + (size_t)h * a.V + pb * COLS;
            float* qd = qs + buf * TCH * Kp;
            float* kd = ks + buf * TCH * Kp;
            float* vd = vs + buf * TCH * COLS;
            float* td = ts + buf * TCH * ROW;
            const float* gates = ROW ? a.table + ((size_t)h * a.n_tokens + first + c0) * ROW : nullptr;
            const float* xr = AUX ? a.aux + (size_t)(first + c0) * a.aux_stride + (size_t)h * a.K : nullptr;
            float* xd = xs + buf * TCH * Kp;
            for (int g = 0; g < GROWS && g * C < nt; ++g) {
                const float* gr = a.group_decay + (size_t)(first + c0 + min((g + 1) * C, nt) - 1) * a.aux_stride + (size_t)h * a.K;
                float* gd = gs + (buf * GROWS + g) * Kp;
                if (a.wide) for (int n = lane * 4; n < a.K; n += 128) copy16_async(gd + n, gr + n);
                else for (int n = lane; n < a.K; n += 32) copy4_async(gd + n, gr + n);
            }
            if (a.wide) {
                if (AUX) copy_rows(xd, Kp, xr, a.aux_stride, a.K / 4, nt, over_k);
                copy_rows(qd, Kp, qr, a.src_stride, a.K / 4, nt, over_k);
                copy_rows(kd, Kp, kr, a.src_stride, a.K / 4, nt, over_k);
                if (v_cols > 0) copy_rows(vd, COLS, vr, a.src_stride, v_cols / 4, nt, over_v);
                if (ROW && !RAW_GATES)
                    for (int i = lane * 4; i < nt * ROW; i += 128) copy16_async(td + i, gates + i);
                return;
            }
            if (ROW && !RAW_GATES)
                for (int i = lane; i < nt * ROW; i += 32) copy4_async(td + i, gates + i);
            for (int tt = 0; tt < nt; ++tt, qr += a.src_stride, kr += a.src_stride, vr += a.src_stride) {
                for (int n = lane; n < a.K; n += 32) {
                    copy4_async(qd + tt * Kp + n, qr + n);
                    copy4_async(kd + tt * Kp + n, kr + n);
                    if (AUX) copy4_async(xd + tt * Kp + n, xr + tt * a.aux_stride + n);
                }
                for (int i = lane; i < v_cols; i += 32) copy4_async(vd + tt * COLS + i, vr + i);
            }
        };
        // the columns behind v's: ones for the normaliser, else nothing; the same in every stage
        for (int i = v_cols + lane; i < COLS; i += 32)
            for (int tt = 0; tt < STAGES * TCH; ++tt) vs[tt * COLS + i] = RULE == RULE_GATED && pb * COLS + i == a.V ? 1.f : 0.f;
        // a last group that is not full is filled up with tokens that change nothing and read nothing
        auto fill_up = [&](int s) {
            const int nt = min(TCH, n_new - s * TCH), buf = s % STAGES;
            for (int tt = nt; tt < (nt + C - 1) / C * C; ++tt) {
                for (int n = lane; n < a.K; n += 32) {
                    qs[(buf * TCH + tt) * Kp + n] = 0.f, ks[(buf * TCH + tt) * Kp + n] = 0.f;
                    if (AUX) xs[(buf * TCH + tt) * Kp + n] = RULE == RULE_DECAYED ? 1.f : 0.f;
                }
                for (int i = lane; i < COLS; i += 32) vs[(buf * TCH + tt) * COLS + i] = 0.f;
                for (int i = lane; i < ROW; i += 32) ts[(buf * TCH + tt) * ROW + i] = i == 0 ? 1.f : 0.f;
            }
        };
        auto write_out = [&](int s) {
            const int c0 = s * TCH, nt = min(TCH, n_new - c0);
            const float* yb = ys + (s & 1) * TCH * COLS;
            const float* tb = ts + s % STAGES * TCH * ROW;
            // lanes over the columns, several tokens side by side where the block has fewer columns than a warp has lanes
            const int per = COLS < 32 ? 32 / COLS : 1, t_in = COLS < 32 ? lane / COLS : 0, c_in = COLS < 32 ? lane % COLS : lane;
            for (int tt = t_in; tt < nt && t_in < per; tt += per) {
                const size_t t = (size_t)(first + c0 + tt);
                for (int i = c_in; i < COLS; i += 32) {
                    const int cc = pb * COLS + i;
                    const float o = yb[tt * COLS + i];
                    if (cc < a.V) a.y[t * (a.H * a.V) + (size_t)h * a.V + cc] = o;
                    else if (cc < a.W) a.den[t * a.H + h] = fmaxf(fabsf(o), tb[tt * ROW + 2]) + 1e-6f;
                }
            }
        };
        copy(0);
        copies_commit();
        if (n_stages > 1) copy(1);
        copies_commit();
        if (RAW_GATES && lane == 0) {
            // one token: its gates on the spot
            const float* row = a.gates + (size_t)first * a.gate_stride + h;
            const float li = log_input(row[a.in_off], a.cap), lf = log_forget(row[a.forget_off], a.cap);
            const float before = m_head[min(pb * COLS, a.W - 1)], m = fmaxf(lf + before, li);      // (m: the same in every column)
            ts[0] = expf(lf + before - m), ts[1] = expf(li - m), ts[2] = expf(-m);
            m_end = m;
        }
        fill_up(0);
        for (int s = 0; s < n_stages; ++s) {
            copies_wait_all_but_one();               // stage s has landed
            __syncthreads();                         // ... for everyone, and everyone is done with the stage before
            if (s > 0) write_out(s - 1);             // (reads the divisors of the stage the next copy goes to)
            __syncwarp();
            if (s + 2 < n_stages) copy(s + 2);
            copies_commit();
            if (s + 2 == n_stages) fill_up(s + 1);
        }
        __syncthreads();
        write_out(n_stages - 1);
        return;
    }

    const int l = tid % LG, col = tid / LG * CPT, c = pb * COLS + col;
    // pair 2 n + r of S: rows (n LG + l) 4 + 2 r and the one behind it
    f2 S[CPT][NP];
#pragma unroll
    for (int p = 0; p < CPT; ++p)
#pragma unroll
        for (int n = 0; n < NR / 4; ++n) {
            const int row = (n * LG + l) * 4;
            const float* s = S_head + (size_t)(c + p) * a.K + row;
            float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
            if (c + p < a.W && a.wide) {
                if (row < a.K) f = *reinterpret_cast<const float4*>(s);
            } else if (c + p < a.W) {
                if (row < a.K) f.x = s[0];
                if (row + 1 < a.K) f.y = s[1];
                if (row + 2 < a.K) f.z = s[2];
                if (row + 3 < a.K) f.w = s[3];
            }
            S[p][2 * n] = f2_of(f.x, f.y);
            S[p][2 * n + 1] = f2_of(f.z, f.w);
        }
    pdl_wait();
    for (int s = 0; s < n_stages; ++s) {
        __syncthreads();
        const int buf = s % STAGES, nt = min(TCH, n_new - s * TCH);
        const ulonglong2* kb = reinterpret_cast<const ulonglong2*>(ks + buf * TCH * Kp) + l;
        const ulonglong2* qb = reinterpret_cast<const ulonglong2*>(qs + buf * TCH * Kp) + l;
        const ulonglong2* xb = reinterpret_cast<const ulonglong2*>(xs + buf * TCH * Kp) + l;
        const ulonglong2* db = reinterpret_cast<const ulonglong2*>(gs + buf * GROWS * Kp) + l;
        const float* vb = vs + buf * TCH * COLS + col;
        const float4* gb = reinterpret_cast<const float4*>(ts + buf * TCH * ROW);      // ROW / 4 a token
        float* yb = ys + (s & 1) * TCH * COLS + col;
        for (int t0 = 0; t0 < nt; t0 += C) {
            if constexpr (Plan::delta) {
                // S^T k and S^T q of the group's tokens, S as it was before them
                constexpr int ND = 2 * C * CPT;
                float dots[ND];
                f2 k[RULE == RULE_DELTA ? C : 1][NP];
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    f2 sk0[CPT], sk1[CPT], sq0[CPT], sq1[CPT];
#pragma unroll
                    for (int p = 0; p < CPT; ++p) sk0[p] = sk1[p] = sq0[p] = sq1[p] = 0ull;
#pragma unroll
                    for (int n = 0; n < NR / 4; ++n) {
                        const ulonglong2 fk = kb[(t0 + j) * (Kp / 4) + n * LG], fq = qb[(t0 + j) * (Kp / 4) + n * LG];
                        if constexpr (RULE == RULE_DELTA) k[j][2 * n] = fk.x, k[j][2 * n + 1] = fk.y;
#pragma unroll
                        for (int p = 0; p < CPT; ++p) {
                            sk0[p] = f2_fma(S[p][2 * n], fk.x, sk0[p]);
                            sk1[p] = f2_fma(S[p][2 * n + 1], fk.y, sk1[p]);
                            sq0[p] = f2_fma(S[p][2 * n], fq.x, sq0[p]);
                            sq1[p] = f2_fma(S[p][2 * n + 1], fq.y, sq1[p]);
                        }
                    }
#pragma unroll
                    for (int p = 0; p < CPT; ++p) {
                        dots[p * 2 * C + j] = f2_sum(f2_add(sk0[p], sk1[p]));
                        dots[p * 2 * C + C + j] = f2_sum(f2_add(sq0[p], sq1[p]));
                    }
                }
                scatter_sum<ND, LG>(dots, lane);
                // the lanes are shared out among the columns; each collects the sums of its own and solves for its u's
                using At = Scattered<ND, LG>;
                constexpr int PER = At::per_lane, STR = At::stride, SHARE = LG / CPT;
                const int mine = CPT > 1 ? l / SHARE : 0;
                float all[2 * C];
#pragma unroll
                for (int i = 0; i < 2 * C; ++i)
                    all[i] = LG == 1 ? dots[i] : __shfl_sync(0xffffffffu, dots[i % PER], mine * (2 * C / PER * STR) + i / PER * STR, LG);
                float u[C], G = 1.f;                 // u_i times the decays of the tokens behind it; the product of all decays
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    const float4 g = gb[(t0 + j) * 3], p0 = gb[(t0 + j) * 3 + 1], p1 = gb[(t0 + j) * 3 + 2];
                    const float kk[3] = {p0.y, p0.w, p1.y}, kq[3] = {p0.z, p1.x, p1.z};
                    if constexpr (RULE == RULE_DELTA) G *= g.x;
                    float b = G * all[j], o = G * all[C + j];
#pragma unroll
                    for (int i = 0; i < j; ++i) {
                        // (channel: the decays in between are in the products and in what is written)
                        if constexpr (RULE == RULE_DELTA) u[i] *= g.x;
                        b = fmaf(kk[(j - i - 1) % 3], u[i], b);
                        o = fmaf(kq[(j - i - 1) % 3], u[i], o);
                    }
                    u[j] = g.y * (vb[(t0 + j) * COLS + mine] - b);
                    o = fmaf(p0.x, u[j], o);
                    if (l % SHARE == 0) yb[(t0 + j) * COLS + mine] = o;
                }
                if constexpr (RULE == RULE_DELTA) {
                    const f2 decay = f2_of(G, G);
#pragma unroll
                    for (int p = 0; p < CPT; ++p)
#pragma unroll
                        for (int n = 0; n < NP; ++n) S[p][n] = f2_mul(decay, S[p][n]);
                } else {
#pragma unroll
                    for (int n = 0; n < NR / 4; ++n) {
                        const ulonglong2 fd = db[t0 / C * (Kp / 4) + n * LG];
#pragma unroll
                        for (int p = 0; p < CPT; ++p) {
                            S[p][2 * n] = f2_mul(fd.x, S[p][2 * n]);
                            S[p][2 * n + 1] = f2_mul(fd.y, S[p][2 * n + 1]);
                        }
                    }
                }
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    f2 uu[CPT];
#pragma unroll
                    for (int p = 0; p < CPT; ++p) {
                        const float up = CPT > 1 ? __shfl_sync(0xffffffffu, u[j], p * SHARE, LG) : u[j];
                        uu[p] = f2_of(up, up);
                    }
#pragma unroll
                    for (int n = 0; n < NR / 4; ++n) {
                        ulonglong2 fw;
                        if constexpr (RULE == RULE_DELTA) fw.x = k[j][2 * n], fw.y = k[j][2 * n + 1];
                        else fw = xb[(t0 + j) * (Kp / 4) + n * LG];
#pragma unroll
                        for (int p = 0; p < CPT; ++p) {
                            S[p][2 * n] = f2_fma(fw.x, uu[p], S[p][2 * n]);
                            S[p][2 * n + 1] = f2_fma(fw.y, uu[p], S[p][2 * n + 1]);
                        }
                    }
                }
            } else {
                float dots[C * CPT];
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    f2 pp[CPT], sq0[CPT], sq1[CPT], decay = 0ull;
                    float put = 1.f;
                    if constexpr (RULE == RULE_GATED) {
                        const float4 g = gb[t0 + j];
                        decay = f2_of(g.x, g.x);
                        put = g.y;
                    }
#pragma unroll
                    for (int p = 0; p < CPT; ++p) {
                        const float pv = put * vb[(t0 + j) * COLS + p];
                        pp[p] = f2_of(pv, pv);
                        sq0[p] = sq1[p] = 0ull;
                    }
#pragma unroll
                    for (int n = 0; n < NR / 4; ++n) {
                        const ulonglong2 fk = kb[(t0 + j) * (Kp / 4) + n * LG], fq = qb[(t0 + j) * (Kp / 4) + n * LG];
                        ulonglong2 fd = {decay, decay};
                        if constexpr (RULE == RULE_DECAYED) fd = xb[(t0 + j) * (Kp / 4) + n * LG];
#pragma unroll
                        for (int p = 0; p < CPT; ++p) {
                            S[p][2 * n] = f2_fma(fk.x, pp[p], f2_mul(fd.x, S[p][2 * n]));
                            S[p][2 * n + 1] = f2_fma(fk.y, pp[p], f2_mul(fd.y, S[p][2 * n + 1]));
                            sq0[p] = f2_fma(S[p][2 * n], fq.x, sq0[p]);
                            sq1[p] = f2_fma(S[p][2 * n + 1], fq.y, sq1[p]);
                        }
                    }
#pragma unroll
                    for (int p = 0; p < CPT; ++p) dots[p * C + j] = f2_sum(f2_add(sq0[p], sq1[p]));
                }
                scatter_sum<C * CPT, LG>(dots, lane);
                using At = Scattered<C * CPT, LG>;
                if (l % At::stride == 0) {
#pragma unroll
                    for (int r = 0; r < At::per_lane; ++r) {
                        const int i = l / At::stride * At::per_lane + r;
                        if (i < C * CPT) yb[(t0 + i % C) * COLS + i / C] = dots[r] * a.q_scale;
                    }
                }
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int p = 0; p < CPT; ++p) {
        if (c + p >= a.W) break;
#pragma unroll
        for (int n = 0; n < NR / 4; ++n) {
            const int row = (n * LG + l) * 4;
            float* s = S_head + (size_t)(c + p) * a.K + row;
            float4 f;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(S[p][2 * n]));
            asm("mov.b64 {%0, %1}, %2;" : "=f"(f.z), "=f"(f.w) : "l"(S[p][2 * n + 1]));
            if (a.wide) {
                if (row < a.K) *reinterpret_cast<float4*>(s) = f;
            } else {
                if (row < a.K) s[0] = f.x;
                if (row + 1 < a.K) s[1] = f.y;
                if (row + 2 < a.K) s[2] = f.z;
                if (row + 3 < a.K) s[3] = f.w;
            }
        }
        if (RAW_GATES && l == 0) m_head[c + p] = m_end;
    }
}

inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

template <int RULE>
int launch_scan(ScanArgs a, int n_entries, bool single, int sm_count, cudaStream_t stream) {
    // Few columns: eight numbers a thread, so that there are warps enough to hide one another's latencies; many: sixteen, so
    // that fewer threads read the same keys and queries.  Portions run best in small blocks, single tokens (one round trip to
    // memory for the whole state) in large ones.
    const int NR = a.K > 256 || (long long)n_entries * a.H * a.W * a.K > 300000 ? 16 : 8;
    int LG = 1;
    while (LG * NR < a.K) LG *= 2;
    const int sms = sm_count > 0 ? sm_count : 148;
    int threads = single ? (NR == 16 ? 128 : 256) : 64;
    while (threads < 4 * LG) threads *= 2;
    while (threads > 32 && threads / 2 >= 4 * LG && (long long)n_entries * a.H * ((a.W + threads / LG - 1) / (threads / LG)) < sms) threads /= 2;
    const int COLS = threads / LG;
    const dim3 grid(n_entries, a.H, (a.W + COLS - 1) / COLS);
    INFERO_REQUIRE(grid.z <= 65535, "memory_scan: %d columns are too many for one launch", a.W);
    a.wide = a.wide && a.V % 4 == 0 && a.v_off % 4 == 0 && COLS % 4 == 0;
    const size_t smem = ScanPlan<RULE>::smem_floats(NR * LG, COLS) * sizeof(float);
#define GO(R, L)                                                                                                       \
    do {                                                                                                               \
        auto k = single ? memory_scan_kernel<RULE, R, L, 1, 1> : memory_scan_kernel<RULE, R, L, GROUP, 1>;             \
        if (smem > 48 * 1024) cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);         \
        /* a portion's blocks run long: started under the kernel in front, they would crowd on the first free SMs */        \
        if (single) launch_pdl(k, grid, dim3(threads + 32), smem, stream, a);                                          \
        else k<<<grid, threads + 32, smem, stream>>>(a);                                                               \
    } while (0)
#define PICK(L)                                                                                                        \
    if (NR == 16) GO(16, L);                                                                                           \
    else GO(8, L);                                                                                                     \
    break
    switch (LG) {
        case 1: PICK(1);
        case 2: PICK(2);
        case 4: PICK(4);
        case 8: PICK(8);
        case 16: PICK(16);
        default: PICK(32);
    }
#undef PICK
#undef GO
    return infero_check_launch("memory_scan");
}

// The rules with decays per channel read three vectors a token, so a thread takes few rows of several columns: what it reads
// serves them all, and a reduction over more lanes costs little more when it carries several columns' sums.  Enough warps to keep
// the schedulers busy come first (INFERO_MEMORY_COLUMNS = 1, 2 or 4 forces the columns of a portion).
inline int forced_columns() {
    static const int v = [] { const char* e = getenv("INFERO_MEMORY_COLUMNS"); return e ? atoi(e) : 0; }();
    return v;
}

template <int RULE>
int launch_channel_scan(ScanArgs a, int n_entries, bool single, int sm_count, cudaStream_t stream) {
    const int NR = a.K <= 128 ? 4 : a.K <= 256 ? 8 : 16, LG = a.K <= 32 ? 8 : a.K <= 64 ? 16 : 32;
    const int sms = sm_count > 0 ? sm_count : 148;
    auto blocks = [&](int cols) { return (long long)n_entries * a.H * ((a.W + cols - 1) / cols); };
    int CPT = 4;
    while (CPT > 1 && blocks(32 / LG * CPT) < 2 * sms) CPT /= 2;         // (blocks of one warp: warps)
    if (single) CPT = CPT == 4 ? 4 : 1;
    else if (forced_columns() == 1 || forced_columns() == 2 || forced_columns() == 4) CPT = forced_columns();
    int threads = single ? 256 : 128;
    while (threads > 32 && threads / 2 / LG * CPT >= 4 && blocks(threads / LG * CPT) * 5 < 4 * sms) threads /= 2;
    const int COLS = threads / LG * CPT;
    const dim3 grid(n_entries, a.H, (a.W + COLS - 1) / COLS);
    INFERO_REQUIRE(grid.z <= 65535, "memory_scan: %d columns are too many for one launch", a.W);
    a.wide = a.wide && a.V % 4 == 0 && a.v_off % 4 == 0 && COLS % 4 == 0;
    const size_t smem = ScanPlan<RULE>::smem_floats(NR * LG, COLS) * sizeof(float);
#define GO(R, L)                                                                                                       \
    do {                                                                                                               \
        auto k = single ? (CPT == 4 ? memory_scan_kernel<RULE, R, L, 1, 4> : memory_scan_kernel<RULE, R, L, 1, 1>)      \
                        : CPT == 4 ? memory_scan_kernel<RULE, R, L, GROUP, 4>                                          \
                        : CPT == 2 ? memory_scan_kernel<RULE, R, L, GROUP, 2> : memory_scan_kernel<RULE, R, L, GROUP, 1>; \
        if (smem > 48 * 1024) cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);         \
        if (single) launch_pdl(k, grid, dim3(threads + 32), smem, stream, a);                                          \
        else k<<<grid, threads + 32, smem, stream>>>(a);                                                               \
    } while (0)
    if (NR == 4 && LG == 8) GO(4, 8);
    else if (NR == 4 && LG == 16) GO(4, 16);
    else if (NR == 4) GO(4, 32);
    else if (NR == 8) GO(8, 32);
    else GO(16, 32);
#undef GO
    return infero_check_launch("memory_scan");
}

// the scans of the other files
int scan_channel(const ScanArgs& a, int n_entries, bool single, int sm_count, cudaStream_t stream);
int scan_decayed(const ScanArgs& a, int n_entries, bool single, int sm_count, cudaStream_t stream);

}  // namespace memory
