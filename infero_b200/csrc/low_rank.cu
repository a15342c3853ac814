// The second half of a product through a narrow middle, with what makes a gate of it, in 32-bit:
//
//   z[t, n] = sum_r a[t, r] w[n, r] (+ bias[n])          a: columns of an input product's 32-bit rows
//   PLAIN    out = z
//   DECAY    out = exp(-exp(a_log[n / per_head]) softplus(z))
//   SIGMOID  out = sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
//
// The middle is a few dozen wide, so the result is bound by its own size; a block makes a tile of tokens by 64 columns,
// both operands transposed in shared memory.  Sums run over r in ascending order, one fused multiply-add each, whatever the
// tile, so a token's numbers do not depend on what else is in the step.
#include "common.cuh"

namespace {

enum : int { LR_PLAIN = 0, LR_DECAY = 1, LR_SIGMOID = 2 };
constexpr int TN = 64, RC = 32, THREADS = 256;      // columns a block makes, how much of the middle is staged at a time

__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

struct LowRankArgs {
    const float* a;
    const void* w;           // [N, R], float32 or bf16
    const float* bias;       // [N] or null
    const float* a_log;      // [N / per_head], DECAY
    float* out;              // [T, N]
    long long a_stride;
    int w_bf16, T, N, R, mode, per_head;
    float inv_tau;
};

__device__ __forceinline__ float finish(const LowRankArgs& p, int n, float z) {
    if (p.bias) z += p.bias[n];
    if (p.mode == LR_DECAY) return expf(-expf(p.a_log[n / p.per_head]) * softplus_f(z));
    if (p.mode == LR_SIGMOID) return expf(-softplus_f(-z) * p.inv_tau);
    return z;
}

// TM tokens: 64 (a thread makes 4 x 4 results) or 8 (2 x 1)
template <int TM>
__global__ void __launch_bounds__(THREADS) low_rank_kernel(const LowRankArgs p) {
    constexpr int PT = TM == 64 ? 4 : 2, PN = TM == 64 ? 4 : 1;
    __shared__ __align__(16) float as[RC][TM + 4], ws[RC][TN + 4];
    pdl_launch_dependents();
    const int tid = threadIdx.x, n0 = blockIdx.x * TN, t0 = blockIdx.y * TM;
    const int tn = TM == 64 ? tid % 16 * 4 : tid % 64, tt = TM == 64 ? tid / 16 * 4 : tid / 64 * 2;
    float acc[PT][PN];
#pragma unroll
    for (int i = 0; i < PT; ++i)
#pragma unroll
        for (int j = 0; j < PN; ++j) acc[i][j] = 0.f;
    bool waited = false;
    for (int r0 = 0; r0 < p.R; r0 += RC) {
        const int nr = min(RC, p.R - r0);
        if (r0) __syncthreads();
        for (int i = tid; i < TN * RC; i += THREADS) {
            const int n = i / RC, r = i % RC;
            float v = 0.f;
            if (r < nr && n0 + n < p.N) {
                const size_t at = (size_t)(n0 + n) * p.R + r0 + r;
                v = p.w_bf16 ? __bfloat162float(((const bf16*)p.w)[at]) : ((const float*)p.w)[at];
            }
            ws[r][n] = v;
        }
        if (!waited) pdl_wait(), waited = true;      // (the weights do not come from a kernel)
        for (int i = tid; i < TM * RC; i += THREADS) {
            const int t = i / RC, r = i % RC;
            as[r][t] = r < nr && t0 + t < p.T ? p.a[(t0 + t) * p.a_stride + r0 + r] : 0.f;
        }
        __syncthreads();
#pragma unroll 4
        for (int r = 0; r < nr; ++r) {
            float x[PT], y[PN];
            if constexpr (TM == 64) {
                const float4 f = *reinterpret_cast<const float4*>(&as[r][tt]), g = *reinterpret_cast<const float4*>(&ws[r][tn]);
                x[0] = f.x, x[1] = f.y, x[2] = f.z, x[3] = f.w;
                y[0] = g.x, y[1] = g.y, y[2] = g.z, y[3] = g.w;
            } else {
                x[0] = as[r][tt], x[1] = as[r][tt + 1], y[0] = ws[r][tn];
            }
#pragma unroll
            for (int i = 0; i < PT; ++i)
#pragma unroll
                for (int j = 0; j < PN; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
        }
    }
    const bool vec = PN == 4 && p.N % 4 == 0;
#pragma unroll
    for (int i = 0; i < PT; ++i) {
        const int t = t0 + tt + i;
        if (t >= p.T) break;
        float* o = p.out + (size_t)t * p.N + n0 + tn;
        float v[PN];
#pragma unroll
        for (int j = 0; j < PN; ++j) v[j] = n0 + tn + j < p.N ? finish(p, n0 + tn + j, acc[i][j]) : 0.f;
        if constexpr (PN == 4) {
            if (vec && n0 + tn + 3 < p.N) {
                *reinterpret_cast<float4*>(o) = make_float4(v[0], v[1], v[2], v[3]);
                continue;
            }
        }
#pragma unroll
        for (int j = 0; j < PN; ++j)
            if (n0 + tn + j < p.N) o[j] = v[j];
    }
}

}  // namespace

extern "C" {

// mode 0: z; 1: exp(-exp(a_log[n / per_head]) softplus(z)); 2: sigmoid(z)^(1 / tau).  out float32 [T, N], 16-byte aligned.
int infero_low_rank(const float* a, long long a_stride, const void* w, int w_dtype, const float* bias, const float* a_log,
                    int per_head, float tau, int mode, float* out, int T, int N, int R, cudaStream_t stream) {
    if (T == 0 || N == 0) return 0;
    INFERO_REQUIRE(R >= 1 && mode >= 0 && mode <= 2, "low_rank: a middle of %d, mode %d", R, mode);
    INFERO_REQUIRE(mode != LR_DECAY || (a_log && per_head >= 1), "low_rank: a decay needs its logarithms");
    INFERO_REQUIRE(mode != LR_SIGMOID || tau > 0.f, "low_rank: tau %g", (double)tau);
    LowRankArgs p = {};
    p.a = a, p.w = w, p.bias = bias, p.a_log = a_log, p.out = out, p.a_stride = a_stride, p.w_bf16 = w_dtype != INFERO_F32;
    p.T = T, p.N = N, p.R = R, p.mode = mode, p.per_head = per_head > 0 ? per_head : 1, p.inv_tau = tau > 0.f ? 1.0f / tau : 1.f;
    const int TM = T > 32 ? 64 : 8;
    const dim3 grid((N + TN - 1) / TN, (T + TM - 1) / TM);
    INFERO_REQUIRE(grid.y <= 65535, "low_rank: %d tokens in one launch", T);
    if (TM == 64) launch_pdl(low_rank_kernel<64>, grid, dim3(THREADS), 0, stream, p);
    else launch_pdl(low_rank_kernel<8>, grid, dim3(THREADS), 0, stream, p);
    return infero_check_launch("low_rank");
}

}  // extern "C"
