// Layers with a norm before and after each sublayer, and a short convolution over time on what a mixer reads.
//
// sandwich_norm, one block per token, does everything between two sublayers in one pass:
//
//   y   = sum of the pending sublayer's result: one 32-bit array or several partial sums (the split-K products of the
//         few-token matrix kernel), plus a bias; or two such results side by side, z = scale * sum_b rms(y_b) * w_b
//   x  += rms(z) * w_post            (w_post null: x += z)
//   h   = rms(x) * w_pre             (the next sublayer's input, or the rows the output product wants; w_pre null: h = x, what
//                                     sublayers without a norm in front read; out null: h is not wanted at all)
//
// with rms(v) = v / sqrt(mean(v^2) + eps).  The weights come as what multiplies (a norm whose stored weight is the
// distance from one is made so at load time).  In steps of single tokens the input convolution below is part of the same
// pass: every token is a request of its own, so its earlier inputs all lie in the request's state.
//
// input_conv: out_t = h_t + sum_j w[j] h_(t - taps + 1 + j) per channel, over the request's new rows and, before them, the
// last taps - 1 inputs its earlier steps left in the state slot (zeros when the request starts); conv_tail moves the
// state on.  h, the weights [taps, d] and the state [taps - 1, d] (oldest first) are 32-bit.
#include "common.cuh"

namespace {

constexpr int MAX_TAPS = 16;

__device__ __forceinline__ void load4(const float* p, float* v) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void store4(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store4(bf16* p, const float* v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}
template <int VEC> __device__ __forceinline__ void load_v(const float* p, float* v) {
    if constexpr (VEC == 4) load4(p, v);
    else v[0] = p[0];
}
template <int VEC, typename T> __device__ __forceinline__ void store_v(T* p, const float* v) {
    if constexpr (VEC == 4) store4(p, v);
    else p[0] = from_f32<T>(v[0]);
}

// Two sums over the block at once, in a fixed order.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* smem64) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    __syncthreads();
    if (lane == 0) { smem64[warp] = a; smem64[32 + warp] = b; }
    __syncthreads();
    a = lane < nwarps ? smem64[lane] : 0.f;
    b = lane < nwarps ? smem64[32 + lane] : 0.f;
    return make_float2(warp_sum(a), warp_sum(b));
}

struct Branch {
    const float* y;          // [splits][rows][d]
    const float* bias;       // [d] or null
    const float* w;          // the branch's own norm weight [d], or null (taken as it is)
    long long split_stride;
    int splits;
};

struct Conv {
    const float* w;          // [taps, d] or null (no convolution in this pass)
    float* state;            // + slot * stride: [taps - 1, d]
    long long state_stride;
    const int* tok_entry;
    const int* entry_slot;
    int taps;
};

// element i (VEC of them) of a branch's row: partial sums in ascending order, eight loads in flight, then the bias
template <int VEC>
__device__ __forceinline__ void branch_row(const Branch& b, size_t row0, int i, float* v) {
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = 0.f;
    for (int s0 = 0; s0 < b.splits; s0 += 8) {
        float t[8][VEC];
#pragma unroll
        for (int s = 0; s < 8; ++s)
            if (s0 + s < b.splits) load_v<VEC>(b.y + (size_t)(s0 + s) * b.split_stride + row0 + i, t[s]);
#pragma unroll
        for (int s = 0; s < 8; ++s)
            if (s0 + s < b.splits) {
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[k] += t[s][k];
            }
    }
    if (b.bias) {
        float t[VEC];
        load_v<VEC>(b.bias + i, t);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] += t[k];
    }
}

template <typename TO, int VEC>
__global__ void __launch_bounds__(1024)
sandwich_norm_kernel(float* __restrict__ x, const Branch b0, const Branch b1, int n_branches, float branch_scale,
                     float branch_eps, const float* __restrict__ w_post, float post_eps, const float* __restrict__ w_pre,
                     float pre_eps, TO* __restrict__ out, const int* __restrict__ rows, int d, const Conv conv) {
    __shared__ float red[64];
    extern __shared__ float buf[];                   // [2][d]; a thread reads back only what it wrote itself
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    const size_t row0 = (size_t)src * d;
    float* xr = x + row0;
    float* z = buf;
    float* y1 = buf + d;
    const int step = blockDim.x * VEC, i0 = threadIdx.x * VEC;
    const float inv_d = 1.0f / (float)d;
    float rz = 1.f;
    if (n_branches > 0) {
        float s0 = 0.f, s1 = 0.f;
        for (int i = i0; i < d; i += step) {
            float v[VEC];
            branch_row<VEC>(b0, row0, i, v);
            store_v<VEC>(z + i, v);
#pragma unroll
            for (int k = 0; k < VEC; ++k) s0 = fmaf(v[k], v[k], s0);
            if (n_branches > 1) {
                branch_row<VEC>(b1, row0, i, v);
                store_v<VEC>(y1 + i, v);
#pragma unroll
                for (int k = 0; k < VEC; ++k) s1 = fmaf(v[k], v[k], s1);
            }
        }
        const float2 s = block_sum2(s0, s1, red);
        if (n_branches > 1 || b0.w) {
            const float r0 = b0.w ? 1.0f / sqrtf(s.x * inv_d + branch_eps) : 1.f;
            const float r1 = n_branches > 1 && b1.w ? 1.0f / sqrtf(s.y * inv_d + branch_eps) : 1.f;
            float sz = 0.f;
            for (int i = i0; i < d; i += step) {
                float v[VEC], w[VEC];
                load_v<VEC>(z + i, v);
                if (b0.w) {
                    load_v<VEC>(b0.w + i, w);
#pragma unroll
                    for (int k = 0; k < VEC; ++k) v[k] = v[k] * r0 * w[k];
                }
                if (n_branches > 1) {
                    float u[VEC];
                    load_v<VEC>(y1 + i, u);
                    if (b1.w) load_v<VEC>(b1.w + i, w);
#pragma unroll
                    for (int k = 0; k < VEC; ++k) v[k] += b1.w ? u[k] * r1 * w[k] : u[k];
                }
#pragma unroll
                for (int k = 0; k < VEC; ++k) {
                    v[k] *= branch_scale;
                    sz = fmaf(v[k], v[k], sz);
                }
                store_v<VEC>(z + i, v);
            }
            if (w_post) rz = 1.0f / sqrtf(block_sum2(sz, 0.f, red).x * inv_d + post_eps);
        } else if (w_post) {
            rz = 1.0f / sqrtf(s.x * inv_d + post_eps);
        }
    }
    float sx = 0.f;
    for (int i = i0; i < d; i += step) {
        float v[VEC];
        load_v<VEC>(xr + i, v);
        if (n_branches > 0) {
            float u[VEC], w[VEC];
            load_v<VEC>(z + i, u);
            if (w_post) {
                load_v<VEC>(w_post + i, w);
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[k] = fmaf(u[k] * rz, w[k], v[k]);
            } else {
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[k] += u[k];
            }
            if (!rows) store_v<VEC>(xr + i, v);
        }
        store_v<VEC>(z + i, v);
#pragma unroll
        for (int k = 0; k < VEC; ++k) sx = fmaf(v[k], v[k], sx);
    }
    if (!out) return;
    const float rx = w_pre ? 1.0f / sqrtf(block_sum2(sx, 0.f, red).x * inv_d + pre_eps) : 1.f;
    TO* orow = out + (size_t)r * d;
    float* tail = conv.w ? conv.state + (long long)conv.entry_slot[conv.tok_entry[src]] * conv.state_stride : nullptr;
    for (int i = i0; i < d; i += step) {
        float h[VEC], w[VEC];
        load_v<VEC>(z + i, h);
        if (w_pre) {
            load_v<VEC>(w_pre + i, w);
#pragma unroll
            for (int k = 0; k < VEC; ++k) h[k] = h[k] * rx * w[k];
        }
        if (conv.w) {
            float acc[VEC], old[VEC];
#pragma unroll
            for (int k = 0; k < VEC; ++k) acc[k] = 0.f;
            for (int j = 0; j < conv.taps - 1; ++j) {
                load_v<VEC>(tail + (size_t)j * d + i, old);
                load_v<VEC>(conv.w + (size_t)j * d + i, w);
#pragma unroll
                for (int k = 0; k < VEC; ++k) acc[k] = fmaf(w[k], old[k], acc[k]);
                if (j > 0) store_v<VEC>(tail + (size_t)(j - 1) * d + i, old);
            }
            if (conv.taps > 1) store_v<VEC>(tail + (size_t)(conv.taps - 2) * d + i, h);
            load_v<VEC>(conv.w + (size_t)(conv.taps - 1) * d + i, w);
#pragma unroll
            for (int k = 0; k < VEC; ++k) h[k] += fmaf(w[k], h[k], acc[k]);
        }
        store_v<VEC>(orow + i, h);
    }
}

// A branch's row as one array, or as partial sums in ascending order with four loads in flight; then the bias.
template <bool PARTIAL>
__device__ __forceinline__ void partial_row(const Branch& b, size_t row0, int i, float* v) {
    load4(b.y + row0 + i, v);
    if (PARTIAL) {
#pragma unroll 4
        for (int s = 1; s < b.splits; ++s) {
            float t[4];
            load4(b.y + (size_t)s * b.split_stride + row0 + i, t);
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] += t[k];
        }
    }
    if (b.bias) {
        float t[4];
        load4(b.bias + i, t);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] += t[k];
    }
}

// The same where a row is at most one vector of four per thread (rows up to 4,096 wide): everything stays in registers, all of
// a row's loads are in flight together, and with more rows than blocks a block has its next row on the way while it works on
// this one.
template <typename TO, int NB, bool PARTIAL>
__global__ void __launch_bounds__(1024)
sandwich_rows_kernel(float* __restrict__ x, const Branch b0, const Branch b1, float branch_scale, float branch_eps,
                     const float* __restrict__ w_post, float post_eps, const float* __restrict__ w_pre, float pre_eps,
                     TO* __restrict__ out, const int* __restrict__ rows, int n_rows, int d, const Conv conv) {
    __shared__ float red[64];
    pdl_launch_dependents();
    const int i = threadIdx.x * 4;
    const bool mine = i < d;
    const float inv_d = 1.0f / (float)d;
    float wq[4] = {0.f, 0.f, 0.f, 0.f}, wp[4] = {0.f, 0.f, 0.f, 0.f};
    if (mine) {
        if (w_pre) load4(w_pre + i, wq);
        if (NB > 0 && w_post) load4(w_post + i, wp);
    }
    pdl_wait();
    float xn[4] = {0.f, 0.f, 0.f, 0.f}, yn[4] = {0.f, 0.f, 0.f, 0.f}, un[4] = {0.f, 0.f, 0.f, 0.f};
    auto fetch = [&](int r) {
        const size_t row0 = (size_t)(rows ? rows[r] : r) * d;
        load4(x + row0 + i, xn);
        if (NB > 0) partial_row<PARTIAL>(b0, row0, i, yn);
        if (NB > 1) partial_row<PARTIAL>(b1, row0, i, un);
    };
    int r = blockIdx.x;
    if (r < n_rows && mine) fetch(r);
    for (; r < n_rows; r += gridDim.x) {
        const int src = rows ? rows[r] : r;
        float v[4], y[4], u[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] = xn[k], y[k] = yn[k], u[k] = un[k];
        if (!PARTIAL && r + gridDim.x < n_rows && mine) fetch(r + gridDim.x);      // (partial sums come in few rows: a block each)
        if (NB > 0) {
            float s0 = 0.f, s1 = 0.f, rz = 1.f;
#pragma unroll
            for (int k = 0; k < 4; ++k) s0 = fmaf(y[k], y[k], s0), s1 = fmaf(u[k], u[k], s1);
            if (NB > 1) {
                const float2 s = block_sum2(s0, s1, red);
                const float r0 = b0.w ? 1.0f / sqrtf(s.x * inv_d + branch_eps) : 1.f, r1 = b1.w ? 1.0f / sqrtf(s.y * inv_d + branch_eps) : 1.f;
                float w0[4] = {1.f, 1.f, 1.f, 1.f}, w1[4] = {1.f, 1.f, 1.f, 1.f};
                if (mine && b0.w) load4(b0.w + i, w0);
                if (mine && b1.w) load4(b1.w + i, w1);
                s0 = 0.f;
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    y[k] = (y[k] * r0 * w0[k] + u[k] * r1 * w1[k]) * branch_scale;
                    s0 = fmaf(y[k], y[k], s0);
                }
            }
            if (w_post) {
                rz = 1.0f / sqrtf(block_sum(s0, red) * inv_d + post_eps);
#pragma unroll
                for (int k = 0; k < 4; ++k) v[k] = fmaf(y[k] * rz, wp[k], v[k]);
            } else {
#pragma unroll
                for (int k = 0; k < 4; ++k) v[k] += y[k];
            }
            if (!rows && mine) store4(x + (size_t)src * d + i, v);
        }
        float sx = 0.f;
#pragma unroll
        for (int k = 0; k < 4; ++k) sx = fmaf(v[k], v[k], sx);
        const float rx = w_pre ? 1.0f / sqrtf(block_sum(sx, red) * inv_d + pre_eps) : 1.f;
        if (!mine || !out) continue;
        if (w_pre) {
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] = v[k] * rx * wq[k];
        }
        if (conv.w) {
            float* tail = conv.state + (long long)conv.entry_slot[conv.tok_entry[src]] * conv.state_stride + i;
            float acc[4] = {0.f, 0.f, 0.f, 0.f}, old[4], w[4];
            for (int j = 0; j < conv.taps - 1; ++j) {
                load4(tail + (size_t)j * d, old);
                load4(conv.w + (size_t)j * d + i, w);
#pragma unroll
                for (int k = 0; k < 4; ++k) acc[k] = fmaf(w[k], old[k], acc[k]);
                if (j > 0) store4(tail + (size_t)(j - 1) * d, old);
            }
            if (conv.taps > 1) store4(tail + (size_t)(conv.taps - 2) * d, v);
            load4(conv.w + (size_t)(conv.taps - 1) * d + i, w);
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] += fmaf(w[k], v[k], acc[k]);
        }
        store4(out + (size_t)r * d + i, v);
    }
}

// Up to four taps: a thread owns four channels of CONV_TOKENS neighbouring tokens and keeps the last three inputs in
// registers, so that a row is read once.
constexpr int CONV_TOKENS = 8;

template <typename TO>
__global__ void __launch_bounds__(256)
input_conv_tile_kernel(const float* __restrict__ h, const float* __restrict__ w, int taps, const float* __restrict__ state,
                       long long state_stride, const int* __restrict__ tok_entry, const int* __restrict__ entry_q_start,
                       const int* __restrict__ entry_slot, TO* __restrict__ out, int n_tokens, int d) {
    pdl_launch_dependents();
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
    float ww[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        ww[j][0] = ww[j][1] = ww[j][2] = ww[j][3] = 0.f;
        if (i < d && j >= 4 - taps) load4(w + (size_t)(j - (4 - taps)) * d + i, ww[j]);
    }
    pdl_wait();
    if (i >= d) return;
    float win[3][4];                                 // the inputs three, two and one token back
    int e = -1;
    const int t0 = blockIdx.y * CONV_TOKENS, t1 = min(n_tokens, t0 + CONV_TOKENS);
    for (int t = t0; t < t1; ++t) {
        if (t == t0 || tok_entry[t] != e) {
            e = tok_entry[t];
            const int first = entry_q_start[e];
            const float* tail = state + (long long)entry_slot[e] * state_stride;
#pragma unroll
            for (int j = 0; j < 3; ++j) {
                const int src = t - first - (3 - j);
                win[j][0] = win[j][1] = win[j][2] = win[j][3] = 0.f;
                if (src >= 0) load4(h + (size_t)(first + src) * d + i, win[j]);
                else if (taps - 1 + src >= 0) load4(tail + (size_t)(taps - 1 + src) * d + i, win[j]);
            }
        }
        float v[4], acc[4];
        load4(h + (size_t)t * d + i, v);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            acc[k] = ww[0][k] * win[0][k];
            acc[k] = fmaf(ww[1][k], win[1][k], acc[k]);
            acc[k] = fmaf(ww[2][k], win[2][k], acc[k]);
            acc[k] = fmaf(ww[3][k], v[k], acc[k]) + v[k];
            win[0][k] = win[1][k], win[1][k] = win[2][k], win[2][k] = v[k];
        }
        store4(out + (size_t)t * d + i, acc);
    }
}

template <typename TO, int VEC>
__global__ void input_conv_kernel(const float* __restrict__ h, const float* __restrict__ w, int taps,
                                  const float* __restrict__ state, long long state_stride, const int* __restrict__ tok_entry,
                                  const int* __restrict__ entry_q_start, const int* __restrict__ entry_slot,
                                  TO* __restrict__ out, int n_tokens, int d) {
    pdl_launch_dependents();
    pdl_wait();
    const int per_row = d / VEC;
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)n_tokens * per_row) return;
    const int t = (int)(idx / per_row), i = (int)(idx % per_row) * VEC;
    const int e = tok_entry[t], first = entry_q_start[e];
    const float* tail = state + (long long)entry_slot[e] * state_stride;
    float acc[VEC], v[VEC], ww[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) acc[k] = 0.f;
    for (int j = 0; j < taps; ++j) {
        const int src = t - first - (taps - 1 - j);
        load_v<VEC>(src >= 0 ? h + (size_t)(first + src) * d + i : tail + (size_t)(taps - 1 + src) * d + i, v);
        load_v<VEC>(w + (size_t)j * d + i, ww);
#pragma unroll
        for (int k = 0; k < VEC; ++k) acc[k] = fmaf(ww[k], v[k], acc[k]);
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) acc[k] += v[k];            // (the last tap's input is the token's own)
    store_v<VEC>(out + (size_t)t * d + i, acc);
}

// A request's tail after n new rows: row r is input n - (taps - 1) + r of the new ones, or what was there before.
__global__ void conv_tail_kernel(const float* __restrict__ h, int h_stride, int taps, float* __restrict__ state,
                                 long long state_stride, const int* __restrict__ entry_q_start,
                                 const int* __restrict__ entry_q_len, const int* __restrict__ entry_slot, int n_entries, int d) {
    pdl_launch_dependents();
    pdl_wait();
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)n_entries * d) return;
    const int e = (int)(idx / d), c = (int)(idx % d);
    const int first = entry_q_start[e], n = entry_q_len[e];
    if (n <= 0) return;
    float* tail = state + (long long)entry_slot[e] * state_stride;
    float keep[MAX_TAPS];
#pragma unroll
    for (int r = 0; r < MAX_TAPS; ++r) {
        if (r < taps - 1) {
            const int src = n - (taps - 1) + r;
            keep[r] = src >= 0 ? h[(size_t)(first + src) * h_stride + c] : tail[(size_t)(n + r) * d + c];
        }
    }
#pragma unroll
    for (int r = 0; r < MAX_TAPS; ++r)
        if (r < taps - 1) tail[(size_t)r * d + c] = keep[r];
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

}  // namespace

extern "C" {

// y0 / y1: `splits` arrays of [rows of x, d] floats, split_stride elements apart (null: absent); bias and w null where there
// is none; w_post null: the sum is added as it is.  rows (null: all): only those rows are worked on and x is left as it
// is.  conv_w (null: none) needs a step of single tokens.
int infero_sandwich_norm(float* x, const float* y0, int splits0, long long stride0, const float* bias0, const float* w0,
                         const float* y1, int splits1, long long stride1, const float* bias1, const float* w1,
                         float branch_scale, float branch_eps, const float* w_post, float post_eps, const float* w_pre,
                         float pre_eps, void* out, int out_dtype, const int* rows, int n_rows, int d, const float* conv_w,
                         int taps, float* state, long long state_stride, const int* tok_entry, const int* entry_slot,
                         cudaStream_t stream) {
    if (n_rows == 0) return 0;
    INFERO_REQUIRE(d > 0 && (size_t)d * 8 <= 200 * 1024, "sandwich_norm: width %d not supported", d);
    INFERO_REQUIRE(w_pre || !conv_w, "sandwich_norm: a convolution needs a normed input");
    INFERO_REQUIRE(out || !w_pre, "sandwich_norm: a norm without a place for its result");
    INFERO_REQUIRE(!y1 || y0, "sandwich_norm: a second branch without a first");
    INFERO_REQUIRE(!conv_w || (taps >= 1 && taps <= MAX_TAPS && !rows), "sandwich_norm: %d taps outside 1..%d", taps, MAX_TAPS);
    const Branch b0 = {y0, bias0, w0, stride0, splits0}, b1 = {y1, bias1, w1, stride1, splits1};
    const Conv conv = {conv_w, state, state_stride, tok_entry, entry_slot, taps};
    const int n_branches = y1 ? 2 : y0 ? 1 : 0;
    const bool vec = d % 4 == 0 && al16(x) && al16(y0) && al16(y1) && al16(bias0) && al16(bias1) && al16(w0) && al16(w1) &&
                     al16(w_post) && al16(w_pre) && al16(out) && al16(conv_w) && al16(state) && state_stride % 4 == 0 &&
                     stride0 % 4 == 0 && stride1 % 4 == 0;
    // (the block size depends on the width alone, so a row's sums are formed in the same order in every step)
    int threads = vec ? (d / 4 + 31) / 32 * 32 : 256;
    if (threads > 1024) threads = 1024;
    const size_t smem = (size_t)d * sizeof(float) * 2;
    if (vec && d <= 4 * threads) {
        static int sms = 0;
        if (!sms) {
            int dev = 0;
            cudaGetDevice(&dev);
            if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0) sms = 148;
        }
        int per_sm = 2048 / threads;
        per_sm = per_sm > 8 ? 8 : per_sm < 1 ? 1 : per_sm;
        const int blocks = n_rows < sms * per_sm ? n_rows : sms * per_sm;
        const bool partial = splits0 > 1 || (y1 && splits1 > 1);
        const int grid = partial ? n_rows : blocks;
#define LAUNCH(TO, NB, P)                                                                                              \
        launch_pdl(sandwich_rows_kernel<TO, NB, P>, dim3(grid), dim3(threads), 0, stream, x, b0, b1, branch_scale, branch_eps, \
                   w_post, post_eps, w_pre, pre_eps, (TO*)out, rows, n_rows, d, conv)
#define PICK(TO)                                                                                                       \
        if (n_branches == 0) LAUNCH(TO, 0, false);                                                                     \
        else if (n_branches == 1 && !w0) { if (partial) LAUNCH(TO, 1, true); else LAUNCH(TO, 1, false); }              \
        else if (n_branches == 2) { if (partial) LAUNCH(TO, 2, true); else LAUNCH(TO, 2, false); }
        if (out_dtype == INFERO_F32) { PICK(float) } else { PICK(bf16) }
#undef PICK
#undef LAUNCH
        if (n_branches != 1 || !w0) return infero_check_launch("sandwich_rows");
    }
#define LAUNCH(TO, V)                                                                                                  \
    do {                                                                                                               \
        auto k = sandwich_norm_kernel<TO, V>;                                                                          \
        if (smem > 48 * 1024) cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);         \
        launch_pdl(k, dim3(n_rows), dim3(threads), smem, stream, x, b0, b1, n_branches, branch_scale, branch_eps, w_post, \
                   post_eps, w_pre, pre_eps, (TO*)out, rows, d, conv);                                                 \
    } while (0)
    if (out_dtype == INFERO_F32) {
        if (vec) LAUNCH(float, 4); else LAUNCH(float, 1);
    } else {
        if (vec) LAUNCH(bf16, 4); else LAUNCH(bf16, 1);
    }
#undef LAUNCH
    return infero_check_launch("sandwich_norm");
}

int infero_conv_tail(const float* h, int h_stride, int taps, float* state, long long state_stride, const int* entry_q_start,
                     const int* entry_q_len, const int* entry_slot, int n_entries, int d, cudaStream_t stream) {
    if (n_entries == 0 || taps <= 1) return 0;
    INFERO_REQUIRE(taps <= MAX_TAPS, "conv_tail: %d taps outside 1..%d", taps, MAX_TAPS);
    const long long per = (long long)n_entries * d;
    launch_pdl(conv_tail_kernel, dim3((unsigned)((per + 255) / 256)), dim3(256), 0, stream, h, h_stride, taps, state, state_stride,
               entry_q_start, entry_q_len, entry_slot, n_entries, d);
    return infero_check_launch("conv_tail");
}

// out = h + conv(h) for every token of the step; then the requests' tails move on.
int infero_input_conv(const float* h, const float* w, int taps, float* state, long long state_stride, const int* tok_entry,
                      const int* entry_q_start, const int* entry_q_len, const int* entry_slot, void* out, int out_dtype,
                      int n_tokens, int n_entries, int d, cudaStream_t stream) {
    if (n_tokens == 0) return 0;
    INFERO_REQUIRE(taps >= 1 && taps <= MAX_TAPS, "input_conv: %d taps outside 1..%d", taps, MAX_TAPS);
    const bool vec = d % 4 == 0 && al16(h) && al16(w) && al16(state) && al16(out) && state_stride % 4 == 0;
    if (vec && taps <= 4) {
        const dim3 tiles((d / 4 + 255) / 256, (n_tokens + CONV_TOKENS - 1) / CONV_TOKENS);
        INFERO_REQUIRE(tiles.y <= 65535, "input_conv: %d tokens in one launch", n_tokens);
        const int threads = d / 4 >= 256 ? 256 : (d / 4 + 31) / 32 * 32;
#define LAUNCH(TO)                                                                                                      \
        launch_pdl(input_conv_tile_kernel<TO>, tiles, dim3(threads), 0, stream, h, w, taps, (const float*)state, state_stride, \
                   tok_entry, entry_q_start, entry_slot, (TO*)out, n_tokens, d)
        if (out_dtype == INFERO_F32) LAUNCH(float); else LAUNCH(bf16);
#undef LAUNCH
        if (infero_check_launch("input_conv_tile")) return 1;
        return infero_conv_tail(h, d, taps, state, state_stride, entry_q_start, entry_q_len, entry_slot, n_entries, d, stream);
    }
    const long long total = (long long)n_tokens * (vec ? d / 4 : d);
    const dim3 grid((unsigned)((total + 255) / 256));
#define LAUNCH(TO, V)                                                                                                  \
    launch_pdl(input_conv_kernel<TO, V>, grid, dim3(256), 0, stream, h, w, taps, (const float*)state, state_stride, tok_entry, \
               entry_q_start, entry_slot, (TO*)out, n_tokens, d)
    if (out_dtype == INFERO_F32) {
        if (vec) LAUNCH(float, 4); else LAUNCH(float, 1);
    } else {
        if (vec) LAUNCH(bf16, 4); else LAUNCH(bf16, 1);
    }
#undef LAUNCH
    if (infero_check_launch("input_conv")) return 1;
    return infero_conv_tail(h, d, taps, state, state_stride, entry_q_start, entry_q_len, entry_slot, n_entries, d, stream);
}

}  // extern "C"
