// The residual stream at a step's start, where more than the token's own embedding goes into it:
//
//   x_t = table[id_t] * scale + bigram[row_t] + pos[p_t]
//   row_t = (id_before * mul_prev + id_t * mul_cur) mod buckets, or `buckets` for a sequence's first token
//
// with either table optional; with a norm of the embedding x_t becomes x_t / sqrt(mean(x_t^2) + eps) * w, and where blocks
// read the residual stream itself its copy in 16 bits (h) is left beside it.  The token before a request's first new one is the last its earlier step brought; it is
// kept per request slot (`previous`).  In steps of single tokens the block that read it also replaces it; in other steps
// a second launch does, after every block has read.  A negative id -(s + 1) stands for the token a sampler left in
// device_tokens[s].
#include "common.cuh"

namespace {

__device__ __forceinline__ int resolve(int id, const int* device_tokens, int vocab) {
    if (id < 0 && device_tokens) id = device_tokens[-id - 1];
    return id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);              // (ids are validated on the host)
}

template <typename TE>
__global__ void embed_compose_kernel(const TE* __restrict__ table, const int* __restrict__ ids,
                                     const int* __restrict__ device_tokens, float* __restrict__ x, int d, int vocab, float scale,
                                     const TE* __restrict__ bigram, long long mul_prev, long long mul_cur, long long buckets,
                                     int* __restrict__ previous, const int* __restrict__ tok_entry,
                                     const int* __restrict__ entry_q_start, const int* __restrict__ entry_slot,
                                     const TE* __restrict__ pos_table, int n_pos, const int* __restrict__ positions, int single,
                                     const float* __restrict__ norm_w, float eps, bf16* __restrict__ h) {
    __shared__ int s_prev;
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int id = resolve(ids[t], device_tokens, vocab);
    const int p = positions[t];
    const TE* brow = nullptr;
    if (bigram) {
        if (threadIdx.x == 0) {
            const int e = tok_entry[t];
            const int slot = entry_slot[e];
            s_prev = t > entry_q_start[e] ? resolve(ids[t - 1], device_tokens, vocab) : previous[slot];
            if (single) previous[slot] = id;
        }
        __syncthreads();
        const long long m = ((long long)s_prev * mul_prev + (long long)id * mul_cur) % buckets;
        const long long row = p == 0 ? buckets : m < 0 ? m + buckets : m;
        brow = bigram + (size_t)row * d;
    }
    const TE* row = table + (size_t)id * d;
    const TE* prow = pos_table ? pos_table + (size_t)min(p, n_pos - 1) * d : nullptr;     // (the host keeps p in range)
    float* o = x + (size_t)t * d;
    float ss = 0.f;
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        float v = to_f32(row[i]) * scale;
        if (brow) v += to_f32(brow[i]);
        if (prow) v += to_f32(prow[i]);
        o[i] = v;
        ss = fmaf(v, v, ss);
        if (h && !norm_w) h[(size_t)t * d + i] = __float2bfloat16_rn(v);
    }
    if (!norm_w) return;
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += blockDim.x) {      // (a thread reads back what it wrote itself)
        const float v = o[i] * r * norm_w[i];
        o[i] = v;
        if (h) h[(size_t)t * d + i] = __float2bfloat16_rn(v);
    }
}

__global__ void keep_previous_kernel(const int* __restrict__ ids, const int* __restrict__ device_tokens, int vocab,
                                     int* __restrict__ previous, const int* __restrict__ entry_q_start,
                                     const int* __restrict__ entry_q_len, const int* __restrict__ entry_slot, int n_entries) {
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x * blockDim.x + threadIdx.x;
    if (e < n_entries && entry_q_len[e] > 0)
        previous[entry_slot[e]] = resolve(ids[entry_q_start[e] + entry_q_len[e] - 1], device_tokens, vocab);
}

}  // namespace

extern "C" {

// single: every request of the step brings one token.  norm_w float32 [d] or null; h bf16 [n_tokens, d] or null.
int infero_embed_compose(const void* table, int dtype, const int* ids, const int* device_tokens, float* x, int n_tokens, int d,
                         int vocab, float scale, const void* bigram, long long mul_prev, long long mul_cur, long long buckets,
                         int* previous, const int* tok_entry, const int* entry_q_start, const int* entry_q_len,
                         const int* entry_slot, int n_entries, const void* pos_table, int n_pos, const int* positions, int single,
                         const float* norm_w, float eps, void* h, cudaStream_t stream) {
    if (n_tokens == 0) return 0;
    INFERO_REQUIRE(d > 0 && vocab > 0, "embed_compose: bad sizes d=%d vocab=%d", d, vocab);
    INFERO_REQUIRE(!bigram || (buckets > 0 && previous), "embed_compose: %lld buckets", buckets);
    INFERO_REQUIRE(!pos_table || n_pos > 0, "embed_compose: an empty position table");
    const int threads = d >= 256 ? 256 : 64;
#define LAUNCH(TE)                                                                                                        \
    launch_pdl(embed_compose_kernel<TE>, dim3(n_tokens), dim3(threads), 0, stream, (const TE*)table, ids, device_tokens, x, d, \
               vocab, scale, (const TE*)bigram, mul_prev, mul_cur, buckets, previous, tok_entry, entry_q_start, entry_slot, \
               (const TE*)pos_table, n_pos, positions, single, norm_w, eps, (bf16*)h)
    if (dtype == INFERO_F32) LAUNCH(float);
    else LAUNCH(bf16);
#undef LAUNCH
    if (bigram && !single)
        launch_pdl(keep_previous_kernel, dim3((n_entries + 127) / 128), dim3(128), 0, stream, ids, device_tokens, vocab, previous,
                   entry_q_start, entry_q_len, entry_slot, n_entries);
    return infero_check_launch("embed_compose");
}

}  // extern "C"
