// The second half of a product through a narrow middle, with what makes a gate of it, in 32-bit:
//
//   z[t, n] = sum_r a[t, r] w[n, r] (+ bias[n])          a: columns of an input product's 32-bit rows
//   PLAIN    out = z
//   DECAY    out = exp(-exp(a_log[n / per_head]) softplus(z))
//   SIGMOID  out = sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau), alone or as the first part of the records [decays | k | q] of a
//            recurrence's scan (channel_memory.cuh), q and k copied from columns of the same rows
//
// The middle is a few dozen wide, so the result is bound by its own size; a block makes a tile of tokens by 64 columns,
// both operands transposed in shared memory.  Sums run over r in ascending order, one fused multiply-add each, whatever the
// tile, so a token's numbers do not depend on what else is in the step.  Two such products of the same step share a launch.
#include "common.cuh"

namespace {

enum : int { LR_PLAIN = 0, LR_DECAY = 1, LR_SIGMOID = 2 };
constexpr int TN = 64, RC = 64, THREADS = 256;      // columns a block makes, how much of the middle is staged at a time

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
    // records: rec [N / per_head, T, 3 row_len], row_len >= per_head (the rows behind are zero); k and q at these columns of qk
    float* rec;
    const float* qk;
    long long qk_stride;
    int q_off, k_off, row_len;
};

// four neighbouring numbers of a row of w, zeros beyond its end
__device__ __forceinline__ void w_quad(const LowRankArgs& p, int n, int r, float* v) {
    const size_t at = (size_t)n * p.R + r;
    if (r + 3 < p.R && (p.R & 3) == 0) {
        if (p.w_bf16) {
            const uint2 u = *reinterpret_cast<const uint2*>((const bf16*)p.w + at);
            v[0] = __uint_as_float(u.x << 16), v[1] = __uint_as_float(u.x & 0xffff0000u);
            v[2] = __uint_as_float(u.y << 16), v[3] = __uint_as_float(u.y & 0xffff0000u);
        } else {
            const float4 f = *reinterpret_cast<const float4*>((const float*)p.w + at);
            v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
        }
        return;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = r + i < p.R ? load_any(p.w, p.w_bf16 ? INFERO_BF16 : INFERO_F32, at + i) : 0.f;
}

// TM tokens: 64 (a thread makes 4 x 4 results) or 8 (2 x 1)
template <int TM>
__global__ void __launch_bounds__(THREADS) low_rank_kernel(const LowRankArgs first, const LowRankArgs second) {
    constexpr int PT = TM == 64 ? 4 : 2, PN = TM == 64 ? 4 : 1;
    __shared__ __align__(16) float as[RC][TM + 4], ws[RC][TN + 4];
    pdl_launch_dependents();
    LowRankArgs p = first;
    if (blockIdx.z) p = second;
    const int tid = threadIdx.x, n0 = blockIdx.x * TN, t0 = blockIdx.y * TM;
    if (n0 >= p.N) return;
    const int tn = TM == 64 ? tid % 16 * 4 : tid % 64, tt = TM == 64 ? tid / 16 * 4 : tid / 64 * 2;
    float acc[PT][PN], bias[PN], rate[PN];
#pragma unroll
    for (int j = 0; j < PN; ++j) {
        const int n = n0 + tn + j;
        bias[j] = p.bias && n < p.N ? p.bias[n] : 0.f;
        rate[j] = p.mode == LR_DECAY && n < p.N ? -expf(p.a_log[n / p.per_head]) : -p.inv_tau;
#pragma unroll
        for (int i = 0; i < PT; ++i) acc[i][j] = 0.f;
    }
    // operands transposed: neighbouring threads take neighbouring rows, four numbers of each
    for (int r0 = 0; r0 < p.R; r0 += RC) {
        const int nr = min(RC, p.R - r0);
        if (r0) __syncthreads();
        for (int r = tid / TN * 4; r < nr; r += THREADS / TN * 4) {
            float v[4] = {0.f, 0.f, 0.f, 0.f};
            const int n = tid % TN;
            if (n0 + n < p.N) w_quad(p, n0 + n, r0 + r, v);
#pragma unroll
            for (int i = 0; i < 4; ++i) ws[r + i][n] = v[i];
        }
        if (!r0) pdl_wait();                         // (the weights do not come from a kernel)
        for (int r = tid / TM * 4; r < nr; r += THREADS / TM * 4) {
            const int t = tid % TM;
            const float* src = p.a + (t0 + t) * p.a_stride + r0 + r;
#pragma unroll
            for (int i = 0; i < 4; ++i) as[r + i][t] = t0 + t < p.T && r + i < nr ? src[i] : 0.f;
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
        for (int j = 0; j < PN; ++j) {
            const float z = acc[i][j] + bias[j];
            v[j] = p.mode == LR_PLAIN ? z : expf(rate[j] * softplus_f(p.mode == LR_DECAY ? z : -z));
        }
        if (p.rec) {
            const float* row = p.qk + t * p.qk_stride;
            if constexpr (PN == 4) {
                const int n = n0 + tn, h = n / p.per_head, c = n - h * p.per_head;
                if (n + 3 < p.N && ((p.per_head | p.q_off | p.k_off | (int)p.qk_stride) & 3) == 0 && c + 4 < p.per_head) {
                    float* r = p.rec + ((size_t)h * p.T + t) * 3 * p.row_len + c;
                    *reinterpret_cast<float4*>(r) = make_float4(v[0], v[1], v[2], v[3]);
                    *reinterpret_cast<float4*>(r + p.row_len) = *reinterpret_cast<const float4*>(row + p.k_off + n);
                    *reinterpret_cast<float4*>(r + 2 * p.row_len) = *reinterpret_cast<const float4*>(row + p.q_off + n);
                    continue;
                }
            }
#pragma unroll
            for (int j = 0; j < PN; ++j) {
                const int n = n0 + tn + j;
                if (n >= p.N) break;
                const int h = n / p.per_head, c = n - h * p.per_head;
                float* r = p.rec + ((size_t)h * p.T + t) * 3 * p.row_len;
                r[c] = v[j], r[p.row_len + c] = row[p.k_off + n], r[2 * p.row_len + c] = row[p.q_off + n];
                if (c == p.per_head - 1)
                    for (int i = p.per_head; i < p.row_len; ++i) r[i] = r[p.row_len + i] = r[2 * p.row_len + i] = 0.f;
            }
            continue;
        }
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

int make_args(LowRankArgs& p, const float* a, long long a_stride, const void* w, int w_dtype, const float* bias, const float* a_log,
              int per_head, float tau, int mode, float* out, int T, int N, int R) {
    INFERO_REQUIRE(R >= 1 && N >= 1 && mode >= 0 && mode <= 2, "low_rank: a middle of %d, %d columns, mode %d", R, N, mode);
    INFERO_REQUIRE(mode != LR_DECAY || (a_log && per_head >= 1), "low_rank: a decay needs its logarithms");
    INFERO_REQUIRE(mode != LR_SIGMOID || tau > 0.f, "low_rank: tau %g", (double)tau);
    INFERO_REQUIRE(((reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15u) == 0, "low_rank: unaligned weights or result");
    p.a = a, p.w = w, p.bias = bias, p.a_log = a_log, p.out = out, p.a_stride = a_stride, p.w_bf16 = w_dtype != INFERO_F32;
    p.T = T, p.N = N, p.R = R, p.mode = mode, p.per_head = per_head > 0 ? per_head : 1, p.inv_tau = tau > 0.f ? 1.0f / tau : 1.f;
    return 0;
}

}  // namespace

extern "C" {

// mode 0: z; 1: exp(-exp(a_log[n / per_head]) softplus(z)); 2: sigmoid(z)^(1 / tau).  out float32 [T, N].  w and out 16-byte
// aligned.  A second product of the same tokens (plain) runs beside the first where N2 > 0.
int infero_low_rank(const float* a, long long a_stride, const void* w, int w_dtype, const float* bias, const float* a_log,
                    int per_head, float tau, int mode, float* out, int T, int N, int R, const float* a2, const void* w2, int w2_dtype,
                    float* out2, int N2, int R2, cudaStream_t stream) {
    if (T == 0) return 0;
    LowRankArgs p = {}, q = {};
    if (make_args(p, a, a_stride, w, w_dtype, bias, a_log, per_head, tau, mode, out, T, N, R)) return 1;
    if (N2 > 0 && make_args(q, a2, a_stride, w2, w2_dtype, nullptr, nullptr, 1, 0.f, LR_PLAIN, out2, T, N2, R2)) return 1;
    const int TM = T > 32 ? 64 : 8, n = N > N2 ? N : N2;
    const dim3 grid((n + TN - 1) / TN, (T + TM - 1) / TM, N2 > 0 ? 2 : 1);
    INFERO_REQUIRE(grid.y <= 65535, "low_rank: %d tokens in one launch", T);
    if (TM == 64) launch_pdl(low_rank_kernel<64>, grid, dim3(THREADS), 0, stream, p, q);
    else launch_pdl(low_rank_kernel<8>, grid, dim3(THREADS), 0, stream, p, q);
    return infero_check_launch("low_rank");
}

// Decays sigmoid(z)^(1 / tau) as records [N / K, T, 3 row_len] with k and q from columns of qk's rows (16-byte aligned).
int infero_low_rank_records(const float* a, long long a_stride, const void* w, int w_dtype, const float* bias, float tau, float* rec,
                            int row_len, const float* qk, long long qk_stride, int q_off, int k_off, int T, int H, int K, int R,
                            cudaStream_t stream) {
    if (T == 0) return 0;
    LowRankArgs p = {};
    if (make_args(p, a, a_stride, w, w_dtype, bias, nullptr, K, tau, LR_SIGMOID, rec, T, H * K, R)) return 1;
    INFERO_REQUIRE(row_len >= K && row_len % 4 == 0 && (reinterpret_cast<uintptr_t>(qk) & 15u) == 0, "low_rank: rows of %d for %d", row_len, K);
    p.rec = rec, p.qk = qk, p.qk_stride = qk_stride, p.q_off = q_off, p.k_off = k_off, p.row_len = row_len;
    const int TM = T > 32 ? 64 : 8;
    const dim3 grid((H * K + TN - 1) / TN, (T + TM - 1) / TM);
    INFERO_REQUIRE(grid.y <= 65535, "low_rank: %d tokens in one launch", T);
    if (TM == 64) launch_pdl(low_rank_kernel<64>, grid, dim3(THREADS), 0, stream, p, p);
    else launch_pdl(low_rank_kernel<8>, grid, dim3(THREADS), 0, stream, p, p);
    return infero_check_launch("low_rank_records");
}

}  // extern "C"
