// The second half of a product through a narrow middle, with what makes a gate of it, in 32-bit:
//
//   z[t, n] = sum_r a[t, r] w[n, r] (+ bias[n])          a: columns of an input product's 32-bit rows
//   PLAIN    out = z
//   DECAY    out = exp(-exp(a_log[n / per_head]) softplus(z))
//   SIGMOID  out = sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau), alone or as the first part of the records [decays | k | q] of a
//            recurrence's scan (channel_memory.cuh), q and k copied from columns of the same rows
//
// A block makes a tile of tokens by 64 columns from rows of both operands in shared memory.  A sum runs over even and odd r side
// by side, each in ascending order, whatever the tile, so a token's numbers do not depend on what else is in the step.  Two such products of the same step share a launch.
#include "outer_memory.cuh"

namespace {

using namespace memory;

enum : int { LR_PLAIN = 0, LR_DECAY = 1, LR_SIGMOID = 2 };
constexpr int TN = 64, RC = 64, THREADS = 256;      // columns a block makes, how much of the middle is staged at a time

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

// TM tokens: 64 (a thread makes 4 tokens by 4 columns, 16 apart) or 8 (2 x 1)
template <int TM>
__global__ void __launch_bounds__(THREADS, 3) low_rank_kernel(const LowRankArgs first, const LowRankArgs second) {
    constexpr bool BIG = TM == 64;
    constexpr int PT = BIG ? 4 : 2, PN = BIG ? 4 : 1, STEP = 16;      // columns of a thread lie this far apart
    __shared__ __align__(16) float as[TM][RC + 4], ws[TN][RC + 4];
    float (*zs)[TN + 4] = reinterpret_cast<float (*)[TN + 4]>(&as[0][0]);       // the sums, in place of a's rows (RC = TN)
    static_assert(RC == TN, "the sums take the place of a's rows");
    pdl_launch_dependents();
    LowRankArgs p = first;
    if (blockIdx.z) p = second;
    const int tid = threadIdx.x, n0 = blockIdx.x * TN, t0 = blockIdx.y * TM;
    if (n0 >= p.N) return;
    const int tn = BIG ? tid % 16 : tid % 64, tt = BIG ? tid / 16 * 4 : tid / 64 * 2;
    f2 acc[PT][PN];
#pragma unroll
    for (int j = 0; j < PN; ++j)
#pragma unroll
        for (int i = 0; i < PT; ++i) acc[i][j] = 0ull;
    const int quad = tid % (RC / 4) * 4;             // a thread brings four neighbouring numbers of a row
    for (int r0 = 0; r0 < p.R; r0 += RC) {
        if (r0) __syncthreads();
        constexpr int ROWS = THREADS / (RC / 4);     // rows of w a pass brings
        float4 wv[TN / ROWS];
#pragma unroll
        for (int k = 0; k < TN / ROWS; ++k) {
            const int n = tid / (RC / 4) + k * ROWS;
            float v[4] = {0.f, 0.f, 0.f, 0.f};
            if (n0 + n < p.N && r0 + quad < p.R) w_quad(p, n0 + n, r0 + quad, v);
            wv[k] = make_float4(v[0], v[1], v[2], v[3]);
        }
#pragma unroll
        for (int k = 0; k < TN / ROWS; ++k) *reinterpret_cast<float4*>(&ws[tid / (RC / 4) + k * ROWS][quad]) = wv[k];
        if (!r0) pdl_wait();                         // (the weights do not come from a kernel)
        constexpr int PASS = THREADS / RC;           // rows of a a pass brings
        const int ar = tid % RC, at = tid / RC;
        const float* src = p.a + (t0 + at) * p.a_stride + r0 + ar;
        float av[TM / PASS];
#pragma unroll
        for (int k = 0; k < TM / PASS; ++k) av[k] = t0 + at + k * PASS < p.T && r0 + ar < p.R ? src[k * PASS * p.a_stride] : 0.f;
#pragma unroll
        for (int k = 0; k < TM / PASS; ++k) as[at + k * PASS][ar] = av[k];
        __syncthreads();
        const int nr = min(RC, (p.R - r0 + 3) & ~3);
#pragma unroll 2
        for (int r = 0; r < nr; r += 4) {
            ulonglong2 x[PT], y[PN];
#pragma unroll
            for (int i = 0; i < PT; ++i) x[i] = *reinterpret_cast<const ulonglong2*>(&as[tt + i][r]);
#pragma unroll
            for (int j = 0; j < PN; ++j) y[j] = *reinterpret_cast<const ulonglong2*>(&ws[tn + j * STEP][r]);
#pragma unroll
            for (int i = 0; i < PT; ++i)
#pragma unroll
                for (int j = 0; j < PN; ++j) acc[i][j] = f2_fma(x[i].y, y[j].y, f2_fma(x[i].x, y[j].x, acc[i][j]));
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < PT; ++i)
#pragma unroll
        for (int j = 0; j < PN; ++j) zs[tt + i][tn + j * STEP] = f2_sum(acc[i][j]);
    __syncthreads();
    // four neighbouring columns of a token at a time, always the same ones
    const int c4 = tid % (TN / 4) * 4, n = n0 + c4, left = p.N - n;
    if (left <= 0) return;
    float bias[4], rate[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const int m = min(n + k, p.N - 1);
        bias[k] = p.bias ? p.bias[m] : 0.f;
        rate[k] = p.mode == LR_DECAY ? -expf(p.a_log[m / p.per_head]) : -p.inv_tau;
    }
    const int h = n / p.per_head, c = n - h * p.per_head;
    const bool whole = left >= 4 && (p.N & 3) == 0 && (!p.rec || (((p.per_head | p.q_off | p.k_off | (int)p.qk_stride) & 3) == 0 &&
                                                           (c + 4 < p.per_head || p.row_len == p.per_head)));
#pragma unroll 1
    for (int i = tid / (TN / 4); i < TM && t0 + i < p.T; i += THREADS / (TN / 4)) {
        const int t = t0 + i;
        const float4 f = *reinterpret_cast<const float4*>(&zs[i][c4]);
        float v[4] = {f.x + bias[0], f.y + bias[1], f.z + bias[2], f.w + bias[3]};
        if (p.mode != LR_PLAIN) {
#pragma unroll
            for (int k = 0; k < 4; ++k) v[k] = expf(rate[k] * softplus_f(p.mode == LR_DECAY ? v[k] : -v[k]));
        }
        if (!p.rec) {
            float* o = p.out + (size_t)t * p.N + n;
            if (whole) *reinterpret_cast<float4*>(o) = make_float4(v[0], v[1], v[2], v[3]);
            else
                for (int k = 0; k < min(4, left); ++k) o[k] = v[k];
            continue;
        }
        const float* row = p.qk + t * p.qk_stride;
        if (whole) {
            float* r = p.rec + ((size_t)h * p.T + t) * 3 * p.row_len + c;
            *reinterpret_cast<float4*>(r) = make_float4(v[0], v[1], v[2], v[3]);
            *reinterpret_cast<float4*>(r + p.row_len) = *reinterpret_cast<const float4*>(row + p.k_off + n);
            *reinterpret_cast<float4*>(r + 2 * p.row_len) = *reinterpret_cast<const float4*>(row + p.q_off + n);
            continue;
        }
        for (int k = 0; k < min(4, left); ++k) {
            const int hh = (n + k) / p.per_head, cc = n + k - hh * p.per_head;
            float* r = p.rec + ((size_t)hh * p.T + t) * 3 * p.row_len;
            r[cc] = v[k], r[p.row_len + cc] = row[p.k_off + n + k], r[2 * p.row_len + cc] = row[p.q_off + n + k];
            if (cc == p.per_head - 1)
                for (int m = p.per_head; m < p.row_len; ++m) r[m] = r[p.row_len + m] = r[2 * p.row_len + m] = 0.f;
        }
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
