// The delta rule with a decay per channel: the convolution, silu, unit vectors and the records of groups of four tokens that the
// scan reads (channel_memory.cuh), and the scan's instances.
#include "channel_memory.cuh"

namespace {

using namespace memory;

// ---- prepare, channel rule -----------------------------------------------------------------------------------------------
struct ChannelArgs {
    PrepareArgs p;           // (u: the values [T, H V]; no table)
    const float* g;          // [T, H K] the decays
    const int* entry_q_len;
    float* rec;              // [H, slots, record]
    int slots, Kp;
};

// the convolution and silu of channels c .. c + VEC of tokens t .. t + nt - 1; zeros beyond
template <int VEC>
__device__ __forceinline__ void conv_group(const PrepareArgs& a, int t, int nt, int first, float* tail, int c, float (*v)[VEC]) {
#pragma unroll
    for (int j = 0; j < GROUP; ++j)
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[j][k] = 0.f;
    if constexpr (VEC == 4) {
        if (a.taps <= 4 && !a.move_tail) {
            Window win;
            window_weights(win, a, c);
            window_start(win, a, t, first, tail, c);
#pragma unroll
            for (int j = 0; j < GROUP; ++j)
                if (j < nt) {
                    float x[4];
                    load4f(a.proj + (size_t)(t + j) * a.proj_stride + a.x_off + c, x);
                    window_next(win, x, v[j]);
                }
            return;
        }
    }
#pragma unroll
    for (int j = 0; j < GROUP; ++j)
        if (j < nt) conv_silu<VEC>(a, t + j, first, tail, c, v[j]);
}

// A warp per (token, unit) where the token starts a group of its request's new tokens; a unit is the q and k of a kv head, worked
// out for every head that reads them, or the v of a head.  In steps of single tokens it also moves its channels' tails on.
template <int VEC, int NV>
__global__ void __launch_bounds__(PREP_WARPS * 32) channel_prepare_kernel(const ChannelArgs ca) {
    const PrepareArgs& a = ca.p;
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * PREP_WARPS + warp;
    const int units = a.G + a.H;
    if (item >= (long long)a.n_tokens * units) return;
    const int t = (int)(item / units), unit = (int)(item % units);
    const int e = a.tok_entry[t], first = a.entry_q_start[e];
    if ((t - first) % GROUP) return;
    const int nt = min(GROUP, first + ca.entry_q_len[e] - t);
    float* tail = a.state + (long long)a.entry_slot[e] * a.state_stride;
    const int HK = a.H * a.K, Kp = ca.Kp, slot = first / GROUP + e + (t - first) / GROUP;
    const int n_rec = a.move_tail ? 1 : GROUP;           // tokens of a record that are read
    if (unit >= a.G) {
        const int h = unit - a.G;
        const size_t U = (size_t)a.H * a.V;
        float* vr = a.u + t * U + (size_t)h * a.V;
        for (int i = lane * VEC; i < a.V; i += 32 * VEC) {
            float v[GROUP][VEC];
            conv_group<VEC>(a, t, nt, first, tail, 2 * a.G * a.K + h * a.V + i, v);
#pragma unroll
            for (int j = 0; j < GROUP; ++j)
                if (j < nt) put<VEC>(vr + j * U + i, v[j]);
        }
        if (lane < n_rec) {
            const float b = lane < nt ? sigmoid_f(a.proj[(size_t)(t + lane) * a.proj_stride + a.step_off + h]) : 0.f;
            ca.rec[((size_t)h * ca.slots + slot) * delta_record(Kp) + Kp + lane * TOKEN_ROW] = b;
        }
        return;
    }
    float q[NV][GROUP][VEC], k[NV][GROUP][VEC];
    float sums[2 * GROUP] = {};
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * 32 + lane) * VEC;
#pragma unroll
        for (int j = 0; j < GROUP; ++j)
#pragma unroll
            for (int r = 0; r < VEC; ++r) q[n][j][r] = k[n][j][r] = 0.f;
        if (i < a.K) {
            conv_group<VEC>(a, t, nt, first, tail, unit * a.K + i, q[n]);
            conv_group<VEC>(a, t, nt, first, tail, (a.G + unit) * a.K + i, k[n]);
#pragma unroll
            for (int j = 0; j < GROUP; ++j)
#pragma unroll
                for (int r = 0; r < VEC; ++r) {
                    sums[j] = fmaf(q[n][j][r], q[n][j][r], sums[j]);
                    sums[GROUP + j] = fmaf(k[n][j][r], k[n][j][r], sums[GROUP + j]);
                }
        }
    }
    scatter_sum<2 * GROUP, 32>(sums, lane);
    const float q_scale = 1.0f / sqrtf((float)a.K);
#pragma unroll
    for (int j = 0; j < GROUP; ++j) {
        const float rq = 1.0f / sqrtf(__shfl_sync(0xffffffffu, sums[0], 4 * j) + 1e-6f) * q_scale;
        const float rk = 1.0f / sqrtf(__shfl_sync(0xffffffffu, sums[0], 4 * (GROUP + j)) + 1e-6f);
#pragma unroll
        for (int n = 0; n < NV; ++n)
#pragma unroll
            for (int r = 0; r < VEC; ++r) q[n][j][r] *= rq, k[n][j][r] *= rk;
    }
    const int per = a.H / a.G;
    for (int h = unit * per; h < (unit + 1) * per; ++h) {
        float* rec = ca.rec + ((size_t)h * ca.slots + slot) * delta_record(Kp);
        float* tok = rec + Kp + TABLE;
        // 0 .. 3: k_j . q_j; then, over the pairs (0,1) (1,2) (2,3) (0,2) (1,3) (0,3), k_i . k_j and k_i . q_j with the decays
        // between
        float dots[16] = {};
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * 32 + lane) * VEC;
            if (i < Kp) {                                // (rows behind K are zero)
                float g[GROUP][VEC];
#pragma unroll
                for (int j = 0; j < GROUP; ++j) {
#pragma unroll
                    for (int r = 0; r < VEC; ++r) g[j][r] = 1.f;
                    if (j < nt && i < a.K) {
                        const float* src = ca.g + (size_t)(t + j) * HK + (size_t)h * a.K + i;
                        if constexpr (VEC == 4) load4f(src, g[j]);
                        else g[j][0] = src[0];
                    }
                }
                float all[VEC], w[GROUP][VEC];           // the decays up to here; D_j k_j
#pragma unroll
                for (int r = 0; r < VEC; ++r) all[r] = 1.f;
#pragma unroll
                for (int j = 0; j < GROUP; ++j) {
                    float gq[VEC], gk[VEC];
#pragma unroll
                    for (int r = 0; r < VEC; ++r) {
                        all[r] *= g[j][r];
                        gq[r] = all[r] * q[n][j][r];
                        gk[r] = all[r] * k[n][j][r];
                        dots[j] = fmaf(k[n][j][r], q[n][j][r], dots[j]);
                        w[j][r] = k[n][j][r];
                    }
#pragma unroll
                    for (int b = 0; b < j; ++b) {        // the tokens before it in the group: pair (b, j), j - b tokens back
                        constexpr int at[GROUP] = {0, 0, 3, 5};
                        const int c = at[j - b] + b;
#pragma unroll
                        for (int r = 0; r < VEC; ++r) {
                            w[b][r] *= g[j][r];
                            dots[4 + c] = fmaf(w[b][r], k[n][j][r], dots[4 + c]);
                            dots[10 + c] = fmaf(w[b][r], q[n][j][r], dots[10 + c]);
                        }
                    }
                    if (j < n_rec) {
                        put<VEC>(tok + j * 3 * Kp + i, gk);
                        put<VEC>(tok + (j * 3 + 1) * Kp + i, gq);
                    }
                }
#pragma unroll
                for (int j = 0; j < GROUP; ++j)
                    if (j < n_rec) put<VEC>(tok + (j * 3 + 2) * Kp + i, w[j]);
                put<VEC>(rec + i, all);
            }
        }
        scatter_sum<16, 32>(dots, lane);                 // value m in lane 2 m
        if (!(lane & 1)) {
            const int m = lane >> 1, c = m < 10 ? m - 4 : m - 10, back = c < 3 ? 1 : c < 5 ? 2 : 3;
            const int j = m < 4 ? m : (back == 1 ? c : back == 2 ? c - 3 : 0) + back;
            if (j < n_rec) rec[Kp + j * TOKEN_ROW + (m < 4 ? 1 : (m < 10 ? 0 : 1) + 2 * back)] = dots[0];
        }
    }
}

}  // namespace

extern "C" {

// Sizes of the delta rule's records: floats of one, and how many a step of n_tokens in n_entries requests needs per head.
int infero_delta_record(int K) { return delta_record(memory::padded_rows(K)); }
int infero_delta_slots(int n_tokens, int n_entries) { return n_tokens / GROUP + n_entries + 1; }
int infero_channel_rows(int K) { return memory::padded_rows(K); }

// v [T, H V] the values and rec [H, slots, record] what the scan reads of every group of four tokens, from the product's rows
// ([q | k | v] at x_off, raw steps at step_off) and the decays g [T, H K].  single: every request of the step brings one token; the
// tails are moved on here then, else by infero_conv_tail.
int infero_channel_prepare(const float* proj, long long proj_stride, int x_off, const float* conv_w, int taps, float* state,
                           long long state_stride, const int* tok_entry, const int* entry_q_start, const int* entry_q_len,
                           const int* entry_slot, float* v, float* rec, int slots, const float* g, int step_off, int n_tokens, int G,
                           int H, int K, int V, int single, cudaStream_t stream) {
    if (n_tokens == 0) return 0;
    INFERO_REQUIRE(taps >= 1 && taps <= MAX_TAPS, "channel_prepare: %d taps outside 1..%d", taps, MAX_TAPS);
    INFERO_REQUIRE(K >= 1 && K <= MAX_K && V >= 1 && G >= 1 && H % G == 0, "channel_prepare: %d heads over %d of %d x %d", H, G, K, V);
    INFERO_REQUIRE(memory::al16(rec), "channel_prepare: unaligned records");
    ChannelArgs c = {};
    PrepareArgs& a = c.p;
    a.proj = proj, a.proj_stride = proj_stride, a.conv_w = conv_w, a.state = state, a.state_stride = state_stride;
    a.tok_entry = tok_entry, a.entry_q_start = entry_q_start, a.entry_slot = entry_slot, a.u = v;
    a.step_off = step_off, a.x_off = x_off, a.taps = taps, a.n_tokens = n_tokens, a.G = G, a.H = H, a.K = K, a.V = V;
    a.CH = 2 * G * K + H * V, a.move_tail = single;
    c.g = g, c.entry_q_len = entry_q_len, c.rec = rec, c.slots = slots, c.Kp = memory::padded_rows(K);
    const long long items = (long long)n_tokens * (G + H);
    const dim3 grid((unsigned)((items + PREP_WARPS - 1) / PREP_WARPS)), block(PREP_WARPS * 32);
    const bool vec = K % 4 == 0 && V % 4 == 0 && proj_stride % 4 == 0 && x_off % 4 == 0 && state_stride % 4 == 0 && al16(proj) &&
                     al16(conv_w) && al16(state) && al16(v) && al16(g);
    if (vec && K <= 128) launch_pdl(channel_prepare_kernel<4, 1>, grid, block, 0, stream, c);
    else if (vec && K <= 256) launch_pdl(channel_prepare_kernel<4, 2>, grid, block, 0, stream, c);
    else if (vec) launch_pdl(channel_prepare_kernel<4, 4>, grid, block, 0, stream, c);
    else if (K <= 128) launch_pdl(channel_prepare_kernel<1, 4>, grid, block, 0, stream, c);
    else launch_pdl(channel_prepare_kernel<1, 16>, grid, block, 0, stream, c);
    return infero_check_launch("channel_prepare");
}

// y [T, H V]: what the heads read out; S [H, V, K] at s_off of the requests' state moves on.
int infero_channel_scan(const float* rec, int slots, const float* v, long long v_stride, float* state, long long state_stride,
                        long long s_off, const int* entry_q_start, const int* entry_q_len, const int* entry_slot, float* y, int n_entries,
                        int single, int H, int K, int V, int sm_count, cudaStream_t stream) {
    return memory::channel_scan<true>(rec, slots, v, v_stride, state, state_stride, s_off, entry_q_start, entry_q_len, entry_slot, y, 1.f,
                                      n_entries, single, H, K, V, sm_count, stream);
}

}  // extern "C"
