// Attention over the paged cache for any batch of tokens: one warp per (token, query head).
//
// For token t of request entry e at position p, head h (kv head h / group):
//   s_j = (q . K[j]) * scale - slope_h * (p - j)   for lo <= j <= p,  lo = window ? max(0, p - window + 1) : 0
//   (slope_h: a per-head distance bias, zero where the caller gives no slopes; or a table by distance,
//   s_j + rel[h][min(p - j, rel_len - 1)]; with a soft cap the scaled product becomes cap tanh(. / cap) before any bias)
//   out = sum_j softmax(s)_j V[j]
// With `cross` head h's weights meet the values of every kv head c, not only its own: out has G * H rows per token, row
// c * H + h, in 32-bit (what a mixing of the heads' weights needs, see head_mix.cu).
// (crates/kernels/src/cu/ops.cu:709-811 is the reference's three-kernel statement; its
// fused decode kernel is ops.cu:1773-2075.  Contiguous head groups: kv head = h / group.)
//
// Keys are visited in ascending order in chunks of 32 aligned to absolute positions, with a
// running maximum and sum (all 32-bit, accurate expf).  The arithmetic done for a token
// depends only on its own position and window, never on how the step was cut or on what
// else is in the batch.  It takes every head size up to 256 and every group size; it is the
// whole of attention on the 32-bit path and the fallback of the bf16 path.
#include "common.cuh"
#include <math_constants.h>

namespace {

constexpr int WARPS = 4;
constexpr int MAX_D = 256;

template <typename T, typename TO>
__global__ void __launch_bounds__(WARPS * 32)
attention_generic_kernel(const T* __restrict__ q, int q_stride, TO* __restrict__ out, int out_stride,
                         const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                         const int* __restrict__ block_table, int max_blocks,
                         const int* __restrict__ tok_entry, const int* __restrict__ positions,
                         int n_tokens, int n_heads, int n_kv, int head_dim, int value_dim, int page_size,
                         int window, float scale, int sink, const float* __restrict__ slopes,
                         const float* __restrict__ rel, int rel_len, int cross, const float* __restrict__ sinks, float softcap) {
    __shared__ float q_s[WARPS][MAX_D];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * WARPS + warp;
    const int rows = cross ? n_heads * n_kv : n_heads;                // results per token
    if (item >= (long long)n_tokens * rows) return;
    const int t = (int)(item / rows), orow_i = (int)(item % rows), h = orow_i % n_heads;
    const int group = n_heads / n_kv;
    const int kvh = h / group, vh = cross ? orow_i / n_heads : kvh;
    const int pos = positions[t];
    const int* table = block_table + (size_t)tok_entry[t] * max_blocks;
    const int lo = window > 0 ? max(0, pos - window + 1) : 0;
    const float slope = slopes ? slopes[h] : 0.f;
    const float* rel_h = rel ? rel + (size_t)h * rel_len : nullptr;

    const T* qrow = q + (size_t)t * q_stride + (size_t)h * head_dim;
    for (int i = lane; i < head_dim; i += 32) q_s[warp][i] = to_f32(qrow[i]);
    __syncwarp();

    // a sink is one more term of the softmax's sum, with score 0 and no value: the running maximum and sum start
    // as if that key had been seen
    // (with learned sinks its score is the head's own number)
    float m = sink ? 0.f : sinks ? sinks[h] : -CUDART_INF_F, l = sink || sinks ? 1.f : 0.f;
    float acc[MAX_D / 32];
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) acc[i] = 0.f;

    for (int j0 = (lo / 32) * 32; j0 <= pos; j0 += 32) {
        const int j = j0 + lane;
        const bool valid = j >= lo && j <= pos;
        long long row = -1;
        float s = -CUDART_INF_F;
        if (valid) {
            const int page = table[j / page_size];
            if (page >= 0) {
                row = ((long long)page * n_kv + kvh) * page_size + (j % page_size);
                const T* kr = k_cache + row * head_dim;
                float d = 0.f;
                for (int i = 0; i < head_dim; ++i) d = fmaf(q_s[warp][i], to_f32(kr[i]), d);
                s = d * scale;
                if (softcap > 0.f) s = softcap * tanhf(s / softcap);
                s -= slope * (float)(pos - j);
                if (rel_h) s += rel_h[min(pos - j, rel_len - 1)];
                row += (long long)(vh - kvh) * page_size;      // from here on: the row of the values
            }
        }
        const float m_new = fmaxf(m, warp_max(s));
        if (m_new == -CUDART_INF_F) continue;         // no readable key in this chunk
        const float p = (row >= 0) ? expf(s - m_new) : 0.f;
        const float corr = expf(m - m_new);          // first chunk: exp(-inf) = 0
        l = l * corr + warp_sum(p);
#pragma unroll
        for (int i = 0; i < MAX_D / 32; ++i) acc[i] *= corr;
        for (int jj = 0; jj < 32; ++jj) {
            const float pj = __shfl_sync(0xffffffffu, p, jj);
            const long long rj = __shfl_sync(0xffffffffu, row, jj);
            if (rj < 0) continue;                      // uniform across the warp
            const T* vr = v_cache + rj * value_dim;
#pragma unroll
            for (int i = 0; i < MAX_D / 32; ++i) {
                const int dd = i * 32 + lane;
                if (dd < value_dim) acc[i] = fmaf(pj, to_f32(vr[dd]), acc[i]);
            }
        }
        m = m_new;
    }
    TO* orow = out + (size_t)t * out_stride + (size_t)orow_i * value_dim;
    const float inv = 1.0f / l;
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) {
        const int dd = i * 32 + lane;
        if (dd < value_dim) orow[dd] = from_f32<TO>(acc[i] * inv);
    }
}

}  // namespace

extern "C" {

// Keys of width head_dim, values of width value_dim (the cache's two arrays have their own row widths); ``sink``:
// the softmax's denominator has one more term exp(0), which carries no value; ``slopes``: float32 [n_heads] or null,
// head h's score loses slopes[h] times the distance between the query and the key; ``rel``: float32 [n_heads, rel_len] or
// null, what a score gains at every distance (the last entry also beyond it); ``cross``: every head meets the values of
// every kv head, out float32 [n_tokens, n_heads * n_kv * value_dim]; ``sinks``: float32 [n_heads] or null, one more term
// exp(sinks[h]) of the denominator; ``softcap`` > 0: scaled scores are soft-capped.
int infero_attention_generic_rel(const void* q, int q_stride, void* out, int out_stride, const void* k_cache,
                                 const void* v_cache, int dtype, const int* block_table, int max_blocks,
                                 const int* tok_entry, const int* positions, int n_tokens, int n_heads,
                                 int n_kv, int head_dim, int value_dim, int page_size, int window, float scale,
                                 int sink, const float* slopes, const float* rel, int rel_len, int cross,
                                 const float* sinks, float softcap, cudaStream_t stream) {
    if (n_tokens == 0) return 0;
    INFERO_REQUIRE(head_dim >= 1 && head_dim <= MAX_D, "attention: head_dim %d outside 1..%d", head_dim, MAX_D);
    INFERO_REQUIRE(value_dim >= 1 && value_dim <= MAX_D, "attention: value width %d outside 1..%d", value_dim, MAX_D);
    INFERO_REQUIRE(n_kv > 0 && n_heads % n_kv == 0, "attention: %d heads not a multiple of %d kv heads", n_heads, n_kv);
    INFERO_REQUIRE(!rel || rel_len >= 1, "attention: an empty table of distances");
    const long long items = (long long)n_tokens * n_heads * (cross ? n_kv : 1);
    const unsigned blocks = (unsigned)((items + WARPS - 1) / WARPS);
#define LAUNCH(T, TO)                                                                                                   \
    attention_generic_kernel<T, TO><<<blocks, WARPS * 32, 0, stream>>>((const T*)q, q_stride, (TO*)out, out_stride,     \
        (const T*)k_cache, (const T*)v_cache, block_table, max_blocks, tok_entry, positions, n_tokens, n_heads, n_kv,   \
        head_dim, value_dim, page_size, window, scale, sink, slopes, rel, rel_len, cross, sinks, softcap)
    if (dtype == INFERO_F32) LAUNCH(float, float);
    else if (cross) LAUNCH(bf16, float);
    else LAUNCH(bf16, bf16);
#undef LAUNCH
    return infero_check_launch("attention_generic");
}

int infero_attention_generic_bias(const void* q, int q_stride, void* out, int out_stride, const void* k_cache,
                                  const void* v_cache, int dtype, const int* block_table, int max_blocks,
                                  const int* tok_entry, const int* positions, int n_tokens, int n_heads,
                                  int n_kv, int head_dim, int value_dim, int page_size, int window, float scale,
                                  int sink, const float* slopes, cudaStream_t stream) {
    return infero_attention_generic_rel(q, q_stride, out, out_stride, k_cache, v_cache, dtype, block_table, max_blocks,
                                        tok_entry, positions, n_tokens, n_heads, n_kv, head_dim, value_dim, page_size,
                                        window, scale, sink, slopes, nullptr, 0, 0, nullptr, 0.f, stream);
}

int infero_attention_generic_ex(const void* q, int q_stride, void* out, int out_stride, const void* k_cache,
                                const void* v_cache, int dtype, const int* block_table, int max_blocks,
                                const int* tok_entry, const int* positions, int n_tokens, int n_heads,
                                int n_kv, int head_dim, int value_dim, int page_size, int window, float scale,
                                int sink, cudaStream_t stream) {
    return infero_attention_generic_bias(q, q_stride, out, out_stride, k_cache, v_cache, dtype, block_table, max_blocks,
                                         tok_entry, positions, n_tokens, n_heads, n_kv, head_dim, value_dim, page_size,
                                         window, scale, sink, nullptr, stream);
}

int infero_attention_generic(const void* q, int q_stride, void* out, int out_stride, const void* k_cache,
                             const void* v_cache, int dtype, const int* block_table, int max_blocks,
                             const int* tok_entry, const int* positions, int n_tokens, int n_heads,
                             int n_kv, int head_dim, int page_size, int window, float scale,
                             cudaStream_t stream) {
    return infero_attention_generic_ex(q, q_stride, out, out_stride, k_cache, v_cache, dtype, block_table, max_blocks,
                                       tok_entry, positions, n_tokens, n_heads, n_kv, head_dim, head_dim, page_size,
                                       window, scale, 0, stream);
}

}  // extern "C"
