// The scan of the recurrences whose state is a matrix per head and whose every row decays on its own (outer_memory.cu has the
// rules with one decay per head).
//
//   delta rule:               S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   gated linear attention:   S <- diag(a) S + k v^T;  o = S^T q
//
// What a token brings besides its value comes as records, packed head by head by the kernel in front, so that a stage of tokens
// is one contiguous piece of memory and one bulk copy:
//
//   delta rule, a record per group of four tokens of a request: [G | table | token 0 | .. | token 3], G [Kp] the product of the
//     group's decays, table 4 x 8 floats (beta; k . q; and, 1, 2 and 3 tokens back in the group, k_back . k and k_back . q with the
//     decays in between), a token [G_j k_j | G_j q_j | D_j k_j] with G_j the product of the decays up
//     to it and D_j that of the tokens behind it.  All factors are at most one; nothing is divided.  A group that is not full is
//     filled up with tokens of zeros.  Request e's groups start at slot (its first row) / 4 + e.
//   gated linear attention, a record per token: [decays | k | q].
//
// Kp is K rounded up to what the lanes hold, the rows behind K zero.  A block owns (request, head, a block of columns); a thread
// holds NR rows of CPT neighbouring columns in registers for the whole portion, so that what it reads of a token serves all of
// them.  Four tokens are taken together: the sums over the lanes of all of them are formed at once, and the delta rule's u's
// follow by forward substitution from the products in the table, the lanes shared out among the columns (a lane keeps its columns
// in an order of its own, the one that it ends up with first, so that the exchanges need no selection).  A helper warp brings
// the stages in, two ahead.  Groups are counted from a request's own first new token: a token's arithmetic does not depend on the
// batch, nor beyond rounding on how its prompt was cut.  Steps of single tokens run the same code in groups of one.
#pragma once
#include "outer_memory.cuh"
#include "tc_common.cuh"

namespace memory {

constexpr int TOKEN_ROW = 8, TABLE = GROUP * TOKEN_ROW;       // floats of a token in a group's table

inline int padded_rows(int K) { return K <= 32 ? 32 : K <= 64 ? 64 : K <= 128 ? 128 : K <= 256 ? 256 : 512; }
__host__ __device__ inline int delta_record(int Kp) { return (1 + 3 * GROUP) * Kp + TABLE; }

struct ChannelScanArgs {
    const float* rec;        // delta: [H, slots, record]; else [H, slots = tokens, 3 Kp]
    const float* v;          // [T, H V] with its own row stride
    float* state;            // + slot * stride + s_off: S [H, V, K]
    const int* entry_q_start;
    const int* entry_q_len;
    const int* entry_slot;
    float* y;                // [T, H V]
    int* err;
    long long v_stride, state_stride, s_off;
    int slots, H, K, V, wide_state, wide_v;
    float q_scale;
};

template <int N> __device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void bulk_copy(void* dst_smem, const void* src, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(tc::smem_u32(dst_smem)),
                 "l"(src), "r"(bytes), "r"(tc::smem_u32(bar)) : "memory");
}

template <bool DELTA, int Kp, int C> struct ChannelPlan {
    static constexpr int TPS = C == 1 ? 1 : Kp > 256 ? 4 : 8;                            // tokens a stage holds
    static constexpr int RING = C == 1 ? 1 : 3;                                     // stages: one at hand, the others on their way
    static constexpr int REC = DELTA ? (1 + 3 * C) * Kp + TABLE : 3 * Kp;                // floats read of a record
    static constexpr int STAGE = DELTA ? TPS / C * REC : TPS * REC;
    // (behind the stages: every warp's u's, written twice, in two turns)
    static size_t smem_bytes(int cols) { return ((size_t)RING * (STAGE + TPS * cols) + (DELTA ? 4 * C * cols : 0)) * sizeof(float); }
};

template <int N> struct Int { static constexpr int value = N; };

template <bool DELTA, int NR, int LG, int C, int CPT>
__global__ void __launch_bounds__(288) channel_scan_kernel(const ChannelScanArgs a) {
    constexpr int Kp = NR * LG, NP = NR / 2, N4 = NR / 4, SHARE = LG / CPT, V4 = 3 * Kp / 4;
    using Plan = ChannelPlan<DELTA, Kp, C>;
    constexpr int TPS = Plan::TPS, REC = Plan::REC;
    extern __shared__ __align__(128) float sm[];
    __shared__ __align__(8) uint64_t full[Plan::RING];
    __shared__ int never;
    const int nc = blockDim.x - 32;                  // threads that hold columns
    const int COLS = nc / LG * CPT;
    float* vs = sm + Plan::RING * Plan::STAGE;           // [Plan::RING][TPS][COLS]
    f2* us = reinterpret_cast<f2*>(vs + Plan::RING * TPS * COLS);         // [2][COLS][C] the u's, twice each
    pdl_launch_dependents();
    const int e = blockIdx.x, h = blockIdx.y, pb = blockIdx.z;
    const int n_new = a.entry_q_len[e];
    if (n_new <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31;
    const int first = a.entry_q_start[e], n_stages = (n_new + TPS - 1) / TPS;
    float* S_head = a.state + (long long)a.entry_slot[e] * a.state_stride + a.s_off + (size_t)h * a.V * a.K;
    if (tid == 0) {
        never = 0;
        for (int i = 0; i < Plan::RING; ++i) tc::mbar_init(&full[i], 1);
        tc::fence_barrier_init();
        tc::fence_proxy_async();
    }
    __syncthreads();
    if (tid >= nc) {
        pdl_wait();
        const int v_cols = max(0, min(COLS, a.V - pb * COLS));
        const float* rec = DELTA ? a.rec + ((size_t)h * a.slots + first / GROUP + e) * delta_record(Kp)
                                 : a.rec + ((size_t)h * a.slots + first) * (3 * Kp);
        const float* v0 = a.v + first * a.v_stride + (size_t)h * a.V + pb * COLS;
        const int chunks = max(1, v_cols / 4);
        auto copy = [&](int s) {
            const int c0 = s * TPS, nt = min(TPS, n_new - c0), buf = s % Plan::RING;
            if (lane == 0) {
                // (in steps of single tokens the front of the one record is all that is wanted)
                const int n = DELTA ? (nt + C - 1) / C * REC : nt * REC;
                tc::mbar_expect_tx(&full[buf], n * 4);
                bulk_copy(sm + buf * Plan::STAGE, rec + (size_t)(DELTA ? c0 / C : c0) * (DELTA ? delta_record(Kp) : REC), n * 4, &full[buf]);
            }
            float* vd = vs + buf * TPS * COLS;
            const float* vr = v0 + c0 * a.v_stride;
            if (a.wide_v) {
                for (int i = lane; i < nt * chunks && v_cols > 0; i += 32)
                    copy16_async(vd + i / chunks * COLS + i % chunks * 4, vr + i / chunks * a.v_stride + i % chunks * 4);
            } else {
                for (int tt = 0; tt < nt; ++tt)
                    for (int i = lane; i < v_cols; i += 32) copy4_async(vd + tt * COLS + i, vr + tt * a.v_stride + i);
            }
        };
        // columns behind v's are zero in every stage; a last group that is not full is filled up with tokens that change
        // nothing and read nothing (the delta rule's records bring them)
        for (int i = v_cols + lane; i < COLS; i += 32)
            for (int tt = 0; tt < Plan::RING * TPS; ++tt) vs[tt * COLS + i] = 0.f;
        auto fill_up = [&](int s) {
            const int nt = min(TPS, n_new - s * TPS), buf = s % Plan::RING;
            for (int tt = nt; tt < (nt + C - 1) / C * C; ++tt) {
                for (int i = lane; i < COLS; i += 32) vs[(buf * TPS + tt) * COLS + i] = 0.f;
                if (!DELTA)
                    for (int i = lane; i < 3 * Kp; i += 32) sm[buf * Plan::STAGE + tt * REC + i] = i < Kp ? 1.f : 0.f;
            }
        };
        constexpr int AHEAD = Plan::RING - 1;
#pragma unroll 1
        for (int s = 0; s < max(1, AHEAD); ++s) {
            if (s < n_stages) copy(s), fill_up(s);
            copies_commit();
        }
        bool ok = true;
        for (int s = 0; s < n_stages; ++s) {
            copies_wait<AHEAD == 0 ? 0 : AHEAD - 1>();           // stage s's values have landed, and so has
            if (ok && !__all_sync(0xffffffffu, tc::mbar_wait(&full[s % Plan::RING], (uint32_t)(s / Plan::RING) & 1u, &never))) {
                ok = false;                          // (its record never came: raise the flag and go on without waiting)
                if (lane == 0) atomicExch(a.err, 9);
            }
            __syncthreads();                         // ... for everyone, and everyone is done with the stage before
            if (AHEAD > 0 && s + AHEAD < n_stages) copy(s + AHEAD), fill_up(s + AHEAD);
            copies_commit();
        }
        if (!ok)                                     // what is still in flight lands before the block's memory goes away
            for (int s = max(0, n_stages - Plan::RING); s < n_stages; ++s) tc::mbar_wait(&full[s % Plan::RING], (uint32_t)(s / Plan::RING) & 1u, &never);
        return;
    }

    const int l = tid % LG, col = tid / LG * CPT, c = pb * COLS + col;
    // The lanes are shared out among the columns: a lane solves (delta rule) and writes the results of column `mine`.  It keeps
    // column p ^ mine in place p, so that what it keeps in an exchange comes first.
    const int mine = l / SHARE, in_share = l % SHARE;
    // pair 2 n + r of S: rows (n LG + l) 4 + 2 r and the one behind it
    f2 S[CPT][NP];
#pragma unroll
    for (int p = 0; p < CPT; ++p)
#pragma unroll
        for (int n = 0; n < N4; ++n) {
            const int row = (n * LG + l) * 4, cc = c + (p ^ mine);
            const float* s = S_head + (size_t)cc * a.K + row;
            float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
            if (cc < a.V && a.wide_state) {
                if (row < a.K) f = *reinterpret_cast<const float4*>(s);
            } else if (cc < a.V) {
                if (row < a.K) f.x = s[0];
                if (row + 1 < a.K) f.y = s[1];
                if (row + 2 < a.K) f.z = s[2];
                if (row + 3 < a.K) f.w = s[3];
            }
            S[p][2 * n] = f2_of(f.x, f.y);
            S[p][2 * n + 1] = f2_of(f.z, f.w);
        }
    pdl_wait();
    const int c_mine = c + mine;
    const size_t y_step = (size_t)a.H * a.V;
    float* yr = a.y + (size_t)first * y_step + (size_t)h * a.V + c_mine;
    // the sums of N values per column over the lanes: column by column to its lanes, then value by value within them
    auto reduce = [&](auto& dots, auto count) {
        constexpr int N = decltype(count)::value;
#pragma unroll
        for (int w = CPT / 2, x = LG / 2; w >= 1; w /= 2, x /= 2)
#pragma unroll
            for (int n = 0; n < w * N; ++n) dots[n] += __shfl_xor_sync(0xffffffffu, dots[n + w * N], x);
        scatter_sum<N, SHARE>(dots, lane);
    };
    int turn = 0;
    for (int s = 0; s < n_stages; ++s) {
        __syncthreads();
        const int buf = s % Plan::RING, nt = min(TPS, n_new - s * TPS);
        const float* vb = vs + buf * TPS * COLS + col;
        for (int t0 = 0; t0 < nt; t0 += C) {
            const float* group = sm + buf * Plan::STAGE + (DELTA ? t0 / C : t0) * REC;
            const ulonglong2* tok = reinterpret_cast<const ulonglong2*>(DELTA ? group + Kp + TABLE : group) + l;
            if constexpr (DELTA) {
                float dots[2 * C * CPT];
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    f2 sk[CPT], sq[CPT];
#pragma unroll
                    for (int n = 0; n < N4; ++n) {
                        const ulonglong2 fk = tok[j * V4 + n * LG], fq = tok[j * V4 + Kp / 4 + n * LG];
#pragma unroll
                        for (int p = 0; p < CPT; ++p) {
                            sk[p] = n ? f2_fma(S[p][2 * n], fk.x, sk[p]) : f2_mul(S[p][0], fk.x);
                            sq[p] = n ? f2_fma(S[p][2 * n], fq.x, sq[p]) : f2_mul(S[p][0], fq.x);
                            sk[p] = f2_fma(S[p][2 * n + 1], fk.y, sk[p]);
                            sq[p] = f2_fma(S[p][2 * n + 1], fq.y, sq[p]);
                        }
                    }
#pragma unroll
                    for (int p = 0; p < CPT; ++p) {
                        dots[p * 2 * C + j] = f2_sum(sk[p]);
                        dots[p * 2 * C + C + j] = f2_sum(sq[p]);
                    }
                }
                reduce(dots, Int<2 * C>());
                using At = Scattered<2 * C, SHARE>;
                float all[2 * C];
#pragma unroll
                for (int i = 0; i < 2 * C; ++i)
                    all[i] = SHARE == 1 ? dots[i] : __shfl_sync(0xffffffffu, dots[i % At::per_lane], i / At::per_lane * At::stride, SHARE);
                const float4* gb = reinterpret_cast<const float4*>(group + Kp);
                float u[C];
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    const float4 p0 = gb[j * 2], p1 = j > 1 ? gb[j * 2 + 1] : make_float4(0.f, 0.f, 0.f, 0.f);
                    const float kk[3] = {p0.z, p1.x, p1.z}, kq[3] = {p0.w, p1.y, p1.w};
                    float b = all[j], o = all[C + j];
#pragma unroll
                    for (int i = 0; i < j; ++i) {
                        b = fmaf(kk[(j - i - 1) % 3], u[i], b);
                        o = fmaf(kq[(j - i - 1) % 3], u[i], o);
                    }
                    u[j] = p0.x * (vb[(t0 + j) * COLS + mine] - b);
                    o = fmaf(p0.y, u[j], o);
                    if (in_share == 0 && c_mine < a.V && t0 + j < nt) yr[(s * TPS + t0 + j) * y_step] = o;
                }
                // every lane needs the u's of all its columns, as pairs
                f2 uu[CPT][C];
                if constexpr (CPT > 1 && C > 1) {
                    f2* ub = us + (turn * COLS + col) * C;
                    turn ^= 1;
                    if (in_share == 0) {
#pragma unroll
                        for (int j = 0; j < C; j += 2)
                            *reinterpret_cast<ulonglong2*>(ub + mine * C + j) = {f2_of(u[j], u[j]), f2_of(u[j + 1], u[j + 1])};
                    }
                    __syncwarp();
#pragma unroll
                    for (int p = 0; p < CPT; ++p)
#pragma unroll
                        for (int j = 0; j < C; j += 2) {
                            const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(ub + (p ^ mine) * C + j);
                            uu[p][j] = f.x, uu[p][j + 1] = f.y;
                        }
                } else {
#pragma unroll
                    for (int p = 0; p < CPT; ++p)
#pragma unroll
                        for (int j = 0; j < C; ++j) {
                            const float up = CPT > 1 ? __shfl_sync(0xffffffffu, u[j], (p ^ mine) * SHARE, LG) : u[j];
                            uu[p][j] = f2_of(up, up);
                        }
                }
                const ulonglong2* gd = reinterpret_cast<const ulonglong2*>(group) + l;
#pragma unroll
                for (int n = 0; n < N4; ++n) {
                    const ulonglong2 fd = gd[n * LG];
#pragma unroll
                    for (int p = 0; p < CPT; ++p) {
                        S[p][2 * n] = f2_mul(fd.x, S[p][2 * n]);
                        S[p][2 * n + 1] = f2_mul(fd.y, S[p][2 * n + 1]);
                    }
                }
#pragma unroll
                for (int j = 0; j < C; ++j)
#pragma unroll
                    for (int n = 0; n < N4; ++n) {
                        const ulonglong2 fw = tok[j * V4 + 2 * (Kp / 4) + n * LG];
#pragma unroll
                        for (int p = 0; p < CPT; ++p) {
                            S[p][2 * n] = f2_fma(fw.x, uu[p][j], S[p][2 * n]);
                            S[p][2 * n + 1] = f2_fma(fw.y, uu[p][j], S[p][2 * n + 1]);
                        }
                    }
            } else {
                float dots[C * CPT];
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    f2 pp[CPT], sq[CPT];
#pragma unroll
                    for (int p = 0; p < CPT; ++p) {
                        const float pv = vb[(t0 + j) * COLS + (p ^ mine)];
                        pp[p] = f2_of(pv, pv);
                    }
#pragma unroll
                    for (int n = 0; n < N4; ++n) {
                        const ulonglong2 fd = tok[j * V4 + n * LG], fk = tok[j * V4 + Kp / 4 + n * LG], fq = tok[j * V4 + 2 * (Kp / 4) + n * LG];
#pragma unroll
                        for (int p = 0; p < CPT; ++p) {
                            S[p][2 * n] = f2_fma(fk.x, pp[p], f2_mul(fd.x, S[p][2 * n]));
                            S[p][2 * n + 1] = f2_fma(fk.y, pp[p], f2_mul(fd.y, S[p][2 * n + 1]));
                            sq[p] = n ? f2_fma(S[p][2 * n], fq.x, sq[p]) : f2_mul(S[p][0], fq.x);
                            sq[p] = f2_fma(S[p][2 * n + 1], fq.y, sq[p]);
                        }
                    }
#pragma unroll
                    for (int p = 0; p < CPT; ++p) dots[p * C + j] = f2_sum(sq[p]);
                }
                reduce(dots, Int<C>());
                using At = Scattered<C, SHARE>;
                if (in_share % At::stride == 0 && c_mine < a.V) {
#pragma unroll
                    for (int r = 0; r < At::per_lane; ++r) {
                        const int j = t0 + in_share / At::stride * At::per_lane + r;
                        if (j < nt) yr[(s * TPS + j) * y_step] = dots[r] * a.q_scale;
                    }
                }
            }
        }
    }
#pragma unroll
    for (int p = 0; p < CPT; ++p) {
        const int cc = c + (p ^ mine);
        if (cc >= a.V) continue;
#pragma unroll
        for (int n = 0; n < N4; ++n) {
            const int row = (n * LG + l) * 4;
            float* s = S_head + (size_t)cc * a.K + row;
            float4 f;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(S[p][2 * n]));
            asm("mov.b64 {%0, %1}, %2;" : "=f"(f.z), "=f"(f.w) : "l"(S[p][2 * n + 1]));
            if (a.wide_state) {
                if (row < a.K) *reinterpret_cast<float4*>(s) = f;
            } else {
                if (row < a.K) s[0] = f.x;
                if (row + 1 < a.K) s[1] = f.y;
                if (row + 2 < a.K) s[2] = f.z;
                if (row + 3 < a.K) s[3] = f.w;
            }
        }
    }
}

// As many columns a thread as leave enough warps to keep the schedulers busy (INFERO_MEMORY_COLUMNS = 1, 2 or 4 forces the columns
// of a portion), and blocks of several warps, which share a stage, as long as there are about as many as multiprocessors.
inline int forced_columns() {
    static const int v = [] { const char* e = getenv("INFERO_MEMORY_COLUMNS"); return e ? atoi(e) : 0; }();
    return v;
}

template <bool DELTA>
int launch_channel_scan(ChannelScanArgs a, int n_entries, bool single, int sm_count, cudaStream_t stream) {
    const int NR = a.K <= 128 ? 4 : a.K <= 256 ? 8 : 16, LG = a.K <= 32 ? 8 : a.K <= 64 ? 16 : 32;
    const int sms = sm_count > 0 ? sm_count : 148;
    auto blocks = [&](int cols) { return (long long)n_entries * a.H * ((a.V + cols - 1) / cols); };
    int CPT = 4;
    while (CPT > 1 && blocks(32 / LG * CPT) < 2 * sms) CPT /= 2;         // (blocks of one warp: warps)
    if (single) CPT = CPT == 4 ? 4 : 1;
    else if (forced_columns() == 1 || forced_columns() == 2 || forced_columns() == 4) CPT = forced_columns();
    int threads = single ? 256 : 128;
    while (threads > 32 && blocks(threads / LG * CPT) * 5 < 4 * sms) threads /= 2;
    const int COLS = threads / LG * CPT;
    const dim3 grid(n_entries, a.H, (a.V + COLS - 1) / COLS);
    INFERO_REQUIRE(grid.z <= 65535, "channel_scan: %d columns are too many for one launch", a.V);
    a.wide_v = a.wide_v && COLS % 4 == 0;
    if (infero_tc_err_flag(&a.err)) return 1;
#define GO(R, L)                                                                                                        \
    do {                                                                                                                \
        auto k = single ? (CPT == 4 ? channel_scan_kernel<DELTA, R, L, 1, 4> : channel_scan_kernel<DELTA, R, L, 1, 1>)   \
                        : CPT == 4 ? channel_scan_kernel<DELTA, R, L, GROUP, 4>                                         \
                        : CPT == 2 ? channel_scan_kernel<DELTA, R, L, GROUP, 2> : channel_scan_kernel<DELTA, R, L, GROUP, 1>; \
        const size_t smem = single ? ChannelPlan<DELTA, R * L, 1>::smem_bytes(COLS) : ChannelPlan<DELTA, R * L, GROUP>::smem_bytes(COLS); \
        if (smem > 48 * 1024) cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);          \
        /* a portion's blocks run long: started under the kernel in front, they would crowd on the first free SMs */         \
        if (single) launch_pdl(k, grid, dim3(threads + 32), smem, stream, a);                                           \
        else k<<<grid, threads + 32, smem, stream>>>(a);                                                                \
    } while (0)
    if (LG == 8) GO(4, 8);
    else if (LG == 16) GO(4, 16);
    else if (NR == 4) GO(4, 32);
    else if (NR == 8) GO(8, 32);
    else GO(16, 32);
#undef GO
    return infero_check_launch("channel_scan");
}

template <bool DELTA>
int channel_scan(const float* rec, int slots, const float* v, long long v_stride, float* state, long long state_stride, long long s_off,
                 const int* entry_q_start, const int* entry_q_len, const int* entry_slot, float* y, float q_scale, int n_entries, int single,
                 int H, int K, int V, int sm_count, cudaStream_t stream) {
    if (n_entries == 0) return 0;
    INFERO_REQUIRE(K >= 1 && K <= MAX_K && V >= 1 && H >= 1 && H <= 65535, "channel_scan: %d heads of %d x %d", H, K, V);
    INFERO_REQUIRE(al16(rec), "channel_scan: unaligned records");
    ChannelScanArgs a = {};
    a.rec = rec, a.v = v, a.state = state, a.entry_q_start = entry_q_start, a.entry_q_len = entry_q_len, a.entry_slot = entry_slot, a.y = y;
    a.v_stride = v_stride, a.state_stride = state_stride, a.s_off = s_off, a.slots = slots, a.H = H, a.K = K, a.V = V, a.q_scale = q_scale;
    a.wide_state = K % 4 == 0 && state_stride % 4 == 0 && s_off % 4 == 0 && al16(state);
    a.wide_v = V % 4 == 0 && v_stride % 4 == 0 && al16(v);
    return launch_channel_scan<DELTA>(a, n_entries, single != 0, sm_count, stream);
}

}  // namespace memory
