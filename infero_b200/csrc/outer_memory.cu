// Recurrences whose state is a matrix per head that every token updates with an outer product, for any batch of requests,
// each with its new tokens and the state its earlier tokens left.  Two rules share the scan:
//
//   delta (the gated delta rule): unit keys k, gates g and beta per head and token,
//       S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//     with  g = exp(-exp(A_log) softplus(a + dt_bias)),  beta = sigmoid(b).
//   gated (the matrix memory of an mLSTM): log gates i and f, a running maximum m (0 at the start),
//       m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k alone
//       o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)
//     with  i = cap tanh(i_raw / cap),  f = log sigmoid(cap tanh(f_raw / cap)).
//     n is one more column of S whose value is always 1.
//
// S is [K, W] per head: K the width of a key, W that of a value (one more in the gated rule).  It is kept with the K
// numbers of a column side by side, [heads, W, K]; the gated rule's m follows as [heads, W], one copy per column.
//
// prepare (delta rule): q, k and v pass a causal convolution over time per channel (zeros before the sequence, the last
//   taps - 1 inputs kept in the request's state) and silu; q and k are made unit vectors per head (1e-6 inside the root),
//   q times K^-1/2.  Beside them are left the products the scan needs within its groups of four tokens: k . q of every token
//   and head, and its k and q with the keys of the tokens before it in its group.
// scan: a block owns (request, head, a block of columns).  A column's K numbers are spread over LG lanes, 8 or 16 each, in
//   registers for the whole portion; tokens are staged sixteen at a time in shared memory by a warp of its own (asynchronous
//   copies, the results of the stage before) while the others work on the stage at hand.  What a token costs is
//   the latency of a reduction over the lanes, so four tokens are taken together: in the delta rule the products of all four
//   keys and queries with the S before them are reduced at once, and the u's follow one after the other from
//       S_j^T x = (g_1 .. g_j) S_0^T x + sum_(i <= j) (g_(i+1) .. g_j) (k_i . x) u_i,
//   exact as it stands; in the gated rule S itself moves token by token and the four read-outs are reduced at once.  Tokens
//   of a request run in order, in groups counted from its own first new token: a token's arithmetic does not depend on the
//   batch, nor beyond rounding on how its prompt was cut.  Steps of single tokens run the same code in groups of one.
// finish: o over its root mean square per head, times a weight, times silu or sigmoid of a gate; a warp per (token, head).
//
// Rules whose every row of S decays on its own are in channel_memory.cuh.
//
// Everything is 32-bit; the result is written in the step's element type.
#include "outer_memory.cuh"

namespace {

using namespace memory;

constexpr int TCH = 16;            // tokens a stage holds
enum : int { RULE_DELTA = 0, RULE_GATED = 1 };

// a token's decay and beta of one head
__device__ __forceinline__ void token_gates(const PrepareArgs& a, int t, int h) {
    const float* row = a.proj + (size_t)t * a.proj_stride;
    float* o = a.table + ((size_t)h * a.n_tokens + t) * DELTA_ROW;
    const float g = expf(-expf(a.a_log[h]) * softplus_f(row[a.decay_off + h] + a.dt_bias[h]));
    *reinterpret_cast<float4*>(o) = make_float4(g, sigmoid_f(row[a.step_off + h]), 0.f, 0.f);
}

template <int VEC>
__global__ void __launch_bounds__(PREP_WARPS * 32) memory_prepare_kernel(const PrepareArgs a) {
    constexpr int NV = MAX_K / (32 * VEC);
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * PREP_WARPS + warp;
    const int units = a.G + a.H;
    if (item >= (long long)a.n_tokens * units) return;
    const int t = (int)(item / units), unit = (int)(item % units);
    const int e = a.tok_entry[t], first = a.entry_q_start[e];
    float* tail = a.state + (long long)a.entry_slot[e] * a.state_stride;
    float* ur = a.u + (size_t)t * a.CH;
    if (unit >= a.G) {                               // a head of v
        const int c0 = 2 * a.G * a.K + (unit - a.G) * a.V;
        for (int i = lane * VEC; i < a.V; i += 32 * VEC) {
            float v[VEC];
            conv_silu<VEC>(a, t, first, tail, c0 + i, v);
            put<VEC>(ur + c0 + i, v);
        }
        if (lane == 0) token_gates(a, t, unit - a.G);
        return;
    }
    const int cq = unit * a.K, ck = a.G * a.K + unit * a.K;
    float q[NV][VEC], k[NV][VEC];
    float sq = 0.f, sk = 0.f, dot = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * 32 + lane) * VEC;
        if (i < a.K) {
            conv_silu<VEC>(a, t, first, tail, cq + i, q[n]);
            conv_silu<VEC>(a, t, first, tail, ck + i, k[n]);
#pragma unroll
            for (int r = 0; r < VEC; ++r) {
                sq = fmaf(q[n][r], q[n][r], sq);
                sk = fmaf(k[n][r], k[n][r], sk);
            }
        }
    }
    const float rq = 1.0f / sqrtf(warp_sum(sq) + 1e-6f) * (1.0f / sqrtf((float)a.K));
    const float rk = 1.0f / sqrtf(warp_sum(sk) + 1e-6f);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * 32 + lane) * VEC;
        if (i < a.K) {
#pragma unroll
            for (int r = 0; r < VEC; ++r) {
                q[n][r] *= rq;
                k[n][r] *= rk;
                dot = fmaf(q[n][r], k[n][r], dot);
            }
            put<VEC>(ur + cq + i, q[n]);
            put<VEC>(ur + ck + i, k[n]);
        }
    }
    const int per = a.H / a.G;                       // the head's products go to every head that reads it: a lane each
    auto gram = [&](int i, float v) {
        for (int h = unit * per + lane; h < (unit + 1) * per; h += 32) a.table[((size_t)h * a.n_tokens + t) * DELTA_ROW + 4 + i] = v;
    };
    gram(0, warp_sum(dot));
    gram(7, 0.f);
    const int back = (t - first) % GROUP;            // (a step of single tokens: none)
    for (int j = 1; j < GROUP; ++j) {
        float ss = 0.f, dk = 0.f, dq = 0.f;
        if (j <= back) {
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int i = (n * 32 + lane) * VEC;
                if (i < a.K) {
                    float p[VEC];
                    conv_silu<VEC>(a, t - j, first, tail, ck + i, p);
#pragma unroll
                    for (int r = 0; r < VEC; ++r) {
                        ss = fmaf(p[r], p[r], ss);
                        dk = fmaf(p[r], k[n][r], dk);
                        dq = fmaf(p[r], q[n][r], dq);
                    }
                }
            }
            const float rp = 1.0f / sqrtf(warp_sum(ss) + 1e-6f);
            dk = warp_sum(dk) * rp;
            dq = warp_sum(dq) * rp;
        }
        gram(2 * j - 1, dk);
        gram(2 * j, dq);
    }
}

// Up to four taps and heads of up to 128 numbers in vectors of four: a warp owns a head of PREP_TOKENS neighbouring tokens, keeps
// the weights and the last three inputs of its channels in registers and reads a row once.
constexpr int PREP_TOKENS = 8;

__global__ void __launch_bounds__(PREP_WARPS * 32) memory_prepare_tile_kernel(const PrepareArgs a) {
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * PREP_WARPS + warp;
    const int units = a.G + a.H;
    const int unit = (int)(item % units);
    const int t0 = (int)(item / units) * PREP_TOKENS, t1 = min(a.n_tokens, t0 + PREP_TOKENS);
    if (t0 >= a.n_tokens) return;                    // (the last block's spare warps)
    const bool keys = unit < a.G;                    // a head of q and k, or a head of v
    const int width = keys ? a.K : a.V, i = lane * 4;
    const bool mine = i < width;
    const int c0 = (keys ? unit * a.K : 2 * a.G * a.K + (unit - a.G) * a.V) + i, c1 = a.G * a.K + c0;
    Window w0 = {}, w1 = {};
    if (mine) {
        window_weights(w0, a, c0);
        if (keys) window_weights(w1, a, c1);
    }
    pdl_wait();
    int e = -1, first = 0;
    const float q_scale = 1.0f / sqrtf((float)a.K);
    const int per = a.H / a.G;
    if (!keys && t0 + lane < t1) token_gates(a, t0 + lane, unit - a.G);
    float back[GROUP - 1][4] = {};                   // the keys one, two and three tokens back
    // a tile that starts within a group goes over the group's keys again, writing nothing
    const int lead = keys ? (t0 - a.entry_q_start[a.tok_entry[t0]]) % GROUP : 0;
    for (int t = t0 - lead; t < t1; ++t) {
        const float* row = a.proj + (size_t)t * a.proj_stride + a.x_off;
        float x0[4] = {0.f, 0.f, 0.f, 0.f}, x1[4] = {0.f, 0.f, 0.f, 0.f}, v0[4], v1[4];
        if (mine) {
            load4f(row + c0, x0);
            if (keys) load4f(row + c1, x1);
        }
        if (a.tok_entry[t] != e) {
            e = a.tok_entry[t];
            first = a.entry_q_start[e];
            const float* tail = a.state + (long long)a.entry_slot[e] * a.state_stride;
            if (mine) {
                window_start(w0, a, t, first, tail, c0);
                if (keys) window_start(w1, a, t, first, tail, c1);
            }
        }
        window_next(w0, x0, v0);
        if (keys) {
            window_next(w1, x1, v1);
            float sq = 0.f, sk = 0.f;
#pragma unroll
            for (int k = 0; k < 4; ++k) sq = fmaf(v0[k], v0[k], sq), sk = fmaf(v1[k], v1[k], sk);
            const float rq = 1.0f / sqrtf(warp_sum(sq) + 1e-6f) * q_scale, rk = 1.0f / sqrtf(warp_sum(sk) + 1e-6f);
            const int in_group = (t - first) % GROUP;
            float p[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int k = 0; k < 4; ++k) v0[k] *= rq, v1[k] *= rk, p[0] = fmaf(v0[k], v1[k], p[0]);
#pragma unroll
            for (int j = 1; j < GROUP; ++j)
                if (j <= in_group) {
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        p[2 * j - 1] = fmaf(back[j - 1][k], v1[k], p[2 * j - 1]);
                        p[2 * j] = fmaf(back[j - 1][k], v0[k], p[2 * j]);
                    }
                }
#pragma unroll
            for (int k = 0; k < 4; ++k) back[2][k] = back[1][k], back[1][k] = back[0][k], back[0][k] = v1[k];
            scatter_sum<8, 32>(p, lane);
            if (t >= t0) {
                if ((lane & 3) == 0)
                    for (int h = unit * per; h < (unit + 1) * per; ++h)
                        a.table[((size_t)h * a.n_tokens + t) * DELTA_ROW + 4 + (lane >> 2)] = p[0];
                if (mine) put<4>(a.u + (size_t)t * a.CH + c1, v1);
            }
        }
        if (mine && t >= t0) put<4>(a.u + (size_t)t * a.CH + c0, v0);
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
    int q_off, k_off, v_off, in_off, forget_off, n_tokens;
    int H, G, K, V, W, wide;
    float q_scale, cap;
};

// The running maximum as pairs (sum of f, largest i + sum of the f behind it), which combine associatively.
struct MaxScan { float F, M; };
__device__ __forceinline__ MaxScan then(MaxScan a, MaxScan b) { return {a.F + b.F, fmaxf(a.M + b.F, b.M)}; }
__device__ __forceinline__ MaxScan warp_scan(MaxScan v, int lane) {
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const MaxScan before = {__shfl_up_sync(0xffffffffu, v.F, o), __shfl_up_sync(0xffffffffu, v.M, o)};
        if (lane >= o) v = then(before, v);
    }
    return v;
}
__device__ __forceinline__ float log_input(float raw, float cap) { return cap * tanhf(raw / cap); }
__device__ __forceinline__ float log_forget(float raw, float cap) { return -softplus_f(-cap * tanhf(raw / cap)); }

// Gated rule, portions: the gates of every token in the table.  A block per (request, head), 256 tokens at a time, the next
// 256 tokens' raw gates on their way meanwhile; the request's m moves on.
constexpr int GATE_THREADS = 256;
__global__ void __launch_bounds__(GATE_THREADS)
memory_gates_kernel(const float* __restrict__ gates, long long gate_stride, int in_off, int forget_off, float cap,
                    float* __restrict__ state, long long state_stride, long long m_off, const int* __restrict__ entry_q_start,
                    const int* __restrict__ entry_q_len, const int* __restrict__ entry_slot, float* __restrict__ table, int n_tokens,
                    int W) {
    __shared__ MaxScan totals[GATE_THREADS / 32];
    __shared__ float s_m;
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int n = entry_q_len[e], first = entry_q_start[e];
    if (n <= 0) return;
    float* m_head = state + (long long)entry_slot[e] * state_stride + m_off + (size_t)h * W;
    float m_run = m_head[0];                         // (the same in every column)
    float ri = 0.f, rf = 0.f;
    auto fetch = [&](int t) {
        if (t >= n) return;
        const float* row = gates + (size_t)(first + t) * gate_stride + h;
        ri = row[in_off];
        rf = row[forget_off];
    };
    fetch(tid);
    for (int c0 = 0; c0 < n; c0 += GATE_THREADS) {
        const int t = c0 + tid;
        const float li = t < n ? log_input(ri, cap) : -INFINITY, lf = t < n ? log_forget(rf, cap) : 0.f;
        fetch(t + GATE_THREADS);
        const MaxScan v = warp_scan({lf, li}, lane);
        if (lane == 31) totals[warp] = v;
        __syncthreads();
        MaxScan before = {0.f, -INFINITY};
        for (int w = 0; w < warp; ++w) before = then(before, totals[w]);
        const float m_warp = fmaxf(before.F + m_run, before.M);      // m in front of this warp's tokens
        const float m = fmaxf(v.F + m_warp, v.M);
        float m_prev = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 0) m_prev = m_warp;
        if (t < n)
            *reinterpret_cast<float4*>(table + ((size_t)h * n_tokens + first + t) * GATED_ROW) =
                make_float4(expf(lf + m_prev - m), expf(li - m), expf(-m), 0.f);
        if (t == min(n, c0 + GATE_THREADS) - 1) s_m = m;
        __syncthreads();
        m_run = s_m;
    }
    for (int c = tid; c < W; c += GATE_THREADS) m_head[c] = m_run;
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
template <int RULE, int NR, int LG, int C>
__global__ void __launch_bounds__(288) memory_scan_kernel(const ScanArgs a) {
    constexpr int Kp = NR * LG, NP = NR / 2, ROW = RULE == RULE_DELTA ? DELTA_ROW : GATED_ROW;
    constexpr bool RAW_GATES = RULE == RULE_GATED && C == 1;
    extern __shared__ __align__(16) float sm[];
    const int nc = blockDim.x - 32;                  // threads that hold columns
    const int COLS = nc / LG;
    float* ks = sm;                                  // [STAGES][TCH][Kp]
    float* qs = ks + STAGES * TCH * Kp;              // [STAGES][TCH][Kp]
    float* ts = qs + STAGES * TCH * Kp;              // [STAGES][TCH][ROW] the tokens' gates
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
            const float* gates = a.table + ((size_t)h * a.n_tokens + first + c0) * ROW;
            if (a.wide) {
                copy_rows(qd, Kp, qr, a.src_stride, a.K / 4, nt, over_k);
                copy_rows(kd, Kp, kr, a.src_stride, a.K / 4, nt, over_k);
                if (v_cols > 0) copy_rows(vd, COLS, vr, a.src_stride, v_cols / 4, nt, over_v);
                if (!RAW_GATES)
                    for (int i = lane * 4; i < nt * ROW; i += 128) copy16_async(td + i, gates + i);
                return;
            }
            if (!RAW_GATES)
                for (int i = lane; i < nt * ROW; i += 32) copy4_async(td + i, gates + i);
            for (int tt = 0; tt < nt; ++tt, qr += a.src_stride, kr += a.src_stride, vr += a.src_stride) {
                for (int n = lane; n < a.K; n += 32) {
                    copy4_async(qd + tt * Kp + n, qr + n);
                    copy4_async(kd + tt * Kp + n, kr + n);
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
                for (int n = lane; n < a.K; n += 32) qs[(buf * TCH + tt) * Kp + n] = 0.f, ks[(buf * TCH + tt) * Kp + n] = 0.f;
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

    const int l = tid % LG, col = tid / LG, c = pb * COLS + col;
    const bool live = c < a.W;
    // pair 2 n + r of S: rows (n LG + l) 4 + 2 r and the one behind it
    f2 S[NP];
#pragma unroll
    for (int n = 0; n < NR / 4; ++n) {
        const int row = (n * LG + l) * 4;
        const float* p = S_head + (size_t)c * a.K + row;
        float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
        if (live && a.wide) {
            if (row < a.K) f = *reinterpret_cast<const float4*>(p);
        } else if (live) {
            if (row < a.K) f.x = p[0];
            if (row + 1 < a.K) f.y = p[1];
            if (row + 2 < a.K) f.z = p[2];
            if (row + 3 < a.K) f.w = p[3];
        }
        S[2 * n] = f2_of(f.x, f.y);
        S[2 * n + 1] = f2_of(f.z, f.w);
    }
    pdl_wait();
    for (int s = 0; s < n_stages; ++s) {
        __syncthreads();
        const int buf = s % STAGES, nt = min(TCH, n_new - s * TCH);
        const ulonglong2* kb = reinterpret_cast<const ulonglong2*>(ks + buf * TCH * Kp) + l;
        const ulonglong2* qb = reinterpret_cast<const ulonglong2*>(qs + buf * TCH * Kp) + l;
        const float* vb = vs + buf * TCH * COLS + col;
        const float4* gb = reinterpret_cast<const float4*>(ts + buf * TCH * ROW);      // ROW / 4 a token
        float* yb = ys + (s & 1) * TCH * COLS + col;
        for (int t0 = 0; t0 < nt; t0 += C) {
            float dots[2 * C];
            if (RULE == RULE_DELTA) {
                // S^T k and S^T q of the group's tokens, S as it was before them
                f2 k[C][NP];
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    f2 sk0 = 0ull, sk1 = 0ull, sq0 = 0ull, sq1 = 0ull;
#pragma unroll
                    for (int n = 0; n < NR / 4; ++n) {
                        const ulonglong2 fk = kb[(t0 + j) * (Kp / 4) + n * LG], fq = qb[(t0 + j) * (Kp / 4) + n * LG];
                        k[j][2 * n] = fk.x, k[j][2 * n + 1] = fk.y;
                        sk0 = f2_fma(S[2 * n], fk.x, sk0);
                        sk1 = f2_fma(S[2 * n + 1], fk.y, sk1);
                        sq0 = f2_fma(S[2 * n], fq.x, sq0);
                        sq1 = f2_fma(S[2 * n + 1], fq.y, sq1);
                    }
                    dots[j] = f2_sum(f2_add(sk0, sk1));
                    dots[C + j] = f2_sum(f2_add(sq0, sq1));
                }
                scatter_sum<2 * C, LG>(dots, lane);
                using At = Scattered<2 * C, LG>;
                float all[2 * C];
#pragma unroll
                for (int i = 0; i < 2 * C; ++i)
                    all[i] = LG == 1 ? dots[i] : __shfl_sync(0xffffffffu, dots[i % At::per_lane], i / At::per_lane * At::stride, LG);
                float u[C], G = 1.f;                 // u_i times the decays of the tokens behind it; the product of all decays
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    const float4 g = gb[(t0 + j) * 3], p0 = gb[(t0 + j) * 3 + 1], p1 = gb[(t0 + j) * 3 + 2];
                    const float kk[3] = {p0.y, p0.w, p1.y}, kq[3] = {p0.z, p1.x, p1.z};
                    G *= g.x;
                    float b = G * all[j], o = G * all[C + j];
#pragma unroll
                    for (int i = 0; i < j; ++i) {
                        u[i] *= g.x;
                        b = fmaf(kk[(j - i - 1) % 3], u[i], b);
                        o = fmaf(kq[(j - i - 1) % 3], u[i], o);
                    }
                    u[j] = g.y * (vb[(t0 + j) * COLS] - b);
                    o = fmaf(p0.x, u[j], o);
                    if (l == 0) yb[(t0 + j) * COLS] = o;
                }
                const f2 decay = f2_of(G, G);
#pragma unroll
                for (int n = 0; n < NP; ++n) S[n] = f2_mul(decay, S[n]);
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    const f2 uu = f2_of(u[j], u[j]);
#pragma unroll
                    for (int n = 0; n < NP; ++n) S[n] = f2_fma(k[j][n], uu, S[n]);
                }
            } else {
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    const float4 g = gb[t0 + j];
                    const float pv = g.y * vb[(t0 + j) * COLS];
                    const f2 decay = f2_of(g.x, g.x), pp = f2_of(pv, pv);
                    f2 sq0 = 0ull, sq1 = 0ull;
#pragma unroll
                    for (int n = 0; n < NR / 4; ++n) {
                        const ulonglong2 fk = kb[(t0 + j) * (Kp / 4) + n * LG], fq = qb[(t0 + j) * (Kp / 4) + n * LG];
                        S[2 * n] = f2_fma(fk.x, pp, f2_mul(decay, S[2 * n]));
                        S[2 * n + 1] = f2_fma(fk.y, pp, f2_mul(decay, S[2 * n + 1]));
                        sq0 = f2_fma(S[2 * n], fq.x, sq0);
                        sq1 = f2_fma(S[2 * n + 1], fq.y, sq1);
                    }
                    dots[j] = f2_sum(f2_add(sq0, sq1));
                }
                scatter_sum<C, LG>(dots, lane);
                using At = Scattered<C, LG>;
                if (l % At::stride == 0) {
#pragma unroll
                    for (int r = 0; r < At::per_lane; ++r) yb[(t0 + l / At::stride * At::per_lane + r) * COLS] = dots[r] * a.q_scale;
                }
            }
        }
    }
    __syncthreads();
    if (!live) return;
#pragma unroll
    for (int n = 0; n < NR / 4; ++n) {
        const int row = (n * LG + l) * 4;
        float* p = S_head + (size_t)c * a.K + row;
        float4 f;
        asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(S[2 * n]));
        asm("mov.b64 {%0, %1}, %2;" : "=f"(f.z), "=f"(f.w) : "l"(S[2 * n + 1]));
        if (a.wide) {
            if (row < a.K) *reinterpret_cast<float4*>(p) = f;
        } else {
            if (row < a.K) p[0] = f.x;
            if (row + 1 < a.K) p[1] = f.y;
            if (row + 2 < a.K) p[2] = f.z;
            if (row + 3 < a.K) p[3] = f.w;
        }
    }
    if (RAW_GATES && l == 0) m_head[c] = m_end;
}

// ---- finish ------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(PREP_WARPS * 32)
memory_finish_kernel(const float* __restrict__ y, const float* __restrict__ den, const float* __restrict__ gate, int gate_stride,
                     int gate_silu, const float* __restrict__ norm_w, int norm_per_head, float eps, float scale, T* __restrict__ out,
                     int out_stride, int n_tokens, int H, int V) {
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * PREP_WARPS + warp;
    if (item >= (long long)n_tokens * H) return;
    const int t = (int)(item / H), h = (int)(item % H);
    const float* yr = y + (size_t)t * H * V + (size_t)h * V;
    const float* gr = gate + (size_t)t * gate_stride + (size_t)h * V;
    const float* w = norm_w + (norm_per_head ? (size_t)h * V : 0);
    T* o = out + (size_t)t * out_stride + (size_t)h * V;
    const float inv = den ? 1.0f / den[(size_t)t * H + h] : 1.0f;
    float ss = 0.f;
    for (int i = lane; i < V; i += 32) {
        const float v = yr[i] * inv;
        ss = fmaf(v, v, ss);
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)V + eps) * inv;
    for (int i = lane; i < V; i += 32) {
        const float g = gr[i];
        o[i] = from_f32<T>(yr[i] * r * w[i] * (gate_silu ? silu_f(g) : sigmoid_f(g)) * scale);
    }
}

__device__ __forceinline__ void store4f(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4f(bf16* p, const float* v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}

// Heads of up to 128 numbers in vectors of four: one round of loads.
template <typename T>
__global__ void __launch_bounds__(PREP_WARPS * 32)
memory_finish_vec_kernel(const float* __restrict__ y, const float* __restrict__ den, const float* __restrict__ gate, int gate_stride,
                         int gate_silu, const float* __restrict__ norm_w, int norm_per_head, float eps, float scale,
                         T* __restrict__ out, int out_stride, int n_tokens, int H, int V) {
    pdl_launch_dependents();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * PREP_WARPS + warp;
    if (item >= (long long)n_tokens * H) return;
    const int t = (int)(item / H), h = (int)(item % H), i = lane * 4;
    const bool mine = i < V;
    float v[4] = {0.f, 0.f, 0.f, 0.f}, g[4] = {0.f, 0.f, 0.f, 0.f}, w[4] = {0.f, 0.f, 0.f, 0.f};
    const float inv = den ? 1.0f / den[(size_t)t * H + h] : 1.0f;
    if (mine) {
        load4f(y + (size_t)t * H * V + (size_t)h * V + i, v);
        load4f(gate + (size_t)t * gate_stride + (size_t)h * V + i, g);
        load4f(norm_w + (norm_per_head ? (size_t)h * V : 0) + i, w);
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) ss = fmaf(v[k] * inv, v[k] * inv, ss);
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)V + eps) * inv;
    if (!mine) return;
#pragma unroll
    for (int k = 0; k < 4; ++k) v[k] = v[k] * r * w[k] * (gate_silu ? silu_f(g[k]) : sigmoid_f(g[k])) * scale;
    store4f(out + (size_t)t * out_stride + (size_t)h * V + i, v);
}

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
    const size_t smem = (size_t)TCH * (STAGES * (2 * NR * LG + DELTA_ROW + COLS) + 2 * COLS) * sizeof(float);
#define GO(R, L)                                                                                                       \
    do {                                                                                                               \
        auto k = single ? memory_scan_kernel<RULE, R, L, 1> : memory_scan_kernel<RULE, R, L, GROUP>;                   \
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

}  // namespace

extern "C" {

int infero_memory_max_key() { return MAX_K; }

// u [T, 2 G K + H V] receives the prepared q, k and v, table [H, T, 12] the gates and the products within
// the scan's groups (see PrepareArgs).  single: every request of the step brings
// one token; the tails are moved on here then, else by infero_conv_tail.
int infero_memory_prepare(const float* proj, long long proj_stride, int x_off, const float* conv_w, int taps, float* state,
                          long long state_stride, const int* tok_entry, const int* entry_q_start, const int* entry_slot,
                          float* u, float* table, const float* a_log, const float* dt_bias, int decay_off, int step_off,
                          int n_tokens, int G, int H, int K, int V, int single, cudaStream_t stream) {
    if (n_tokens == 0) return 0;
    INFERO_REQUIRE(taps >= 1 && taps <= MAX_TAPS, "memory_prepare: %d taps outside 1..%d", taps, MAX_TAPS);
    INFERO_REQUIRE(K >= 1 && K <= MAX_K && V >= 1 && G >= 1 && H % G == 0, "memory_prepare: %d heads over %d of %d x %d", H, G, K, V);
    PrepareArgs a = {};
    a.proj = proj, a.proj_stride = proj_stride, a.conv_w = conv_w, a.state = state, a.state_stride = state_stride;
    a.tok_entry = tok_entry, a.entry_q_start = entry_q_start, a.entry_slot = entry_slot, a.u = u, a.table = table;
    a.a_log = a_log, a.dt_bias = dt_bias, a.decay_off = decay_off, a.step_off = step_off;
    a.x_off = x_off, a.taps = taps, a.n_tokens = n_tokens, a.G = G, a.H = H, a.K = K, a.V = V, a.CH = 2 * G * K + H * V;
    a.move_tail = single;
    const long long items = (long long)n_tokens * (G + H);
    const dim3 grid((unsigned)((items + PREP_WARPS - 1) / PREP_WARPS));
    const bool vec = K % 4 == 0 && V % 4 == 0 && proj_stride % 4 == 0 && x_off % 4 == 0 && state_stride % 4 == 0 && al16(proj) &&
                     al16(conv_w) && al16(state) && al16(u);
    if (vec && !single && taps <= 4 && K <= 128 && V <= 128) {
        const long long tiles = (long long)((n_tokens + PREP_TOKENS - 1) / PREP_TOKENS) * (G + H);
        launch_pdl(memory_prepare_tile_kernel, dim3((unsigned)((tiles + PREP_WARPS - 1) / PREP_WARPS)), dim3(PREP_WARPS * 32), 0, stream, a);
        return infero_check_launch("memory_prepare_tile");
    }
    if (vec) launch_pdl(memory_prepare_kernel<4>, grid, dim3(PREP_WARPS * 32), 0, stream, a);
    else launch_pdl(memory_prepare_kernel<1>, grid, dim3(PREP_WARPS * 32), 0, stream, a);
    return infero_check_launch("memory_prepare");
}

// table [H, n_tokens, 4] receives every token's gates; the requests' m at m_off of their state [H, W] moves on.
int infero_memory_gates(const float* gates, long long gate_stride, int in_off, int forget_off, float cap, float* state,
                        long long state_stride, long long m_off, const int* entry_q_start, const int* entry_q_len,
                        const int* entry_slot, float* table, int n_tokens, int n_entries, int H, int W, cudaStream_t stream) {
    if (n_entries == 0) return 0;
    INFERO_REQUIRE(H >= 1 && H <= 65535 && cap > 0.f, "memory_gates: %d heads, cap %g", H, (double)cap);
    launch_pdl(memory_gates_kernel, dim3(n_entries, H), dim3(GATE_THREADS), 0, stream, gates, gate_stride, in_off, forget_off, cap, state,
               state_stride, m_off, entry_q_start, entry_q_len, entry_slot, table, n_tokens, W);
    return infero_check_launch("memory_gates");
}

// rule 0 (delta): src and table as infero_memory_prepare leaves them; rule 1 (gated): src the product's rows, table as
// infero_memory_gates leaves it, or, in steps of single tokens, gates the product's rows.
// single: every request of the step brings one token.
int infero_memory_scan(int rule, const float* src, long long src_stride, int q_off, int k_off, int v_off, const float* table,
                       int n_tokens, const float* gates, long long gate_stride, int in_off, int forget_off, float cap,
                       float q_scale, float* state, long long state_stride, long long s_off, const int* entry_q_start,
                       const int* entry_q_len, const int* entry_slot, float* y, float* den, int n_entries, int single, int H,
                       int G, int K, int V, int sm_count, cudaStream_t stream) {
    if (n_entries == 0) return 0;
    INFERO_REQUIRE(K >= 1 && K <= MAX_K && V >= 1 && G >= 1 && H % G == 0 && H <= 65535, "memory_scan: %d heads over %d of %d x %d", H, G, K, V);
    ScanArgs a = {};
    a.src = src, a.gates = gates, a.table = table, a.state = state, a.n_tokens = n_tokens;
    a.entry_q_start = entry_q_start, a.entry_q_len = entry_q_len, a.entry_slot = entry_slot, a.y = y, a.den = den;
    a.src_stride = src_stride, a.gate_stride = gate_stride, a.state_stride = state_stride, a.s_off = s_off;
    a.q_off = q_off, a.k_off = k_off, a.v_off = v_off, a.in_off = in_off, a.forget_off = forget_off;
    a.H = H, a.G = G, a.K = K, a.V = V, a.W = rule == RULE_GATED ? V + 1 : V;
    a.q_scale = q_scale, a.cap = cap;
    a.wide = K % 4 == 0 && src_stride % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && state_stride % 4 == 0 && s_off % 4 == 0 &&
             al16(src) && al16(state) && al16(table);
    INFERO_REQUIRE(table || (rule == RULE_GATED && single && gates), "memory_scan: no gates");
    return rule == RULE_GATED ? launch_scan<RULE_GATED>(a, n_entries, single != 0, sm_count, stream)
                              : launch_scan<RULE_DELTA>(a, n_entries, single != 0, sm_count, stream);
}

// out[t, h V + i] = v / sqrt(mean over the head of v^2 + eps) * w_i * act(gate[t, h V + i]) * scale with v = y / den (den null:
// y); w of V numbers shared by the heads, or (norm_per_head) of H V; act silu or sigmoid.
int infero_memory_finish(const float* y, const float* den, const float* gate, int gate_stride, int gate_silu, const float* norm_w,
                         int norm_per_head, float eps, float scale, void* out, int out_stride, int dtype, int n_tokens, int H, int V,
                         cudaStream_t stream) {
    if (n_tokens == 0) return 0;
    const long long items = (long long)n_tokens * H;
    const dim3 grid((unsigned)((items + PREP_WARPS - 1) / PREP_WARPS));
    if (V % 4 == 0 && V <= 128 && gate_stride % 4 == 0 && out_stride % 4 == 0 && al16(y) && al16(gate) && al16(norm_w) && al16(out)) {
        if (dtype == INFERO_F32)
            launch_pdl(memory_finish_vec_kernel<float>, grid, dim3(PREP_WARPS * 32), 0, stream, y, den, gate, gate_stride, gate_silu, norm_w,
                       norm_per_head, eps, scale, (float*)out, out_stride, n_tokens, H, V);
        else
            launch_pdl(memory_finish_vec_kernel<bf16>, grid, dim3(PREP_WARPS * 32), 0, stream, y, den, gate, gate_stride, gate_silu, norm_w,
                       norm_per_head, eps, scale, (bf16*)out, out_stride, n_tokens, H, V);
        return infero_check_launch("memory_finish");
    }
    if (dtype == INFERO_F32)
        launch_pdl(memory_finish_kernel<float>, grid, dim3(PREP_WARPS * 32), 0, stream, y, den, gate, gate_stride, gate_silu, norm_w,
                   norm_per_head, eps, scale, (float*)out, out_stride, n_tokens, H, V);
    else
        launch_pdl(memory_finish_kernel<bf16>, grid, dim3(PREP_WARPS * 32), 0, stream, y, den, gate, gate_stride, gate_silu, norm_w,
                   norm_per_head, eps, scale, (bf16*)out, out_stride, n_tokens, H, V);
    return infero_check_launch("memory_finish");
}

}  // extern "C"
