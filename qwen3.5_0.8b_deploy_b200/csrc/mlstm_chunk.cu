// Chunk-128 mLSTM prefill on tcgen05 tensor cores.
//
// With F_t the running sum of the log forget gates inside a chunk, a_s = i_s - F_s, m_0 the running maximum at the chunk
// start and M_t = max(m_0, a_1 .. a_t), the token recurrence (mlstm.cu) is m_t = F_t + M_t and
//     num_t = e^{m_0 - M_t} S_0^T q_t + sum_{s <= t} e^{a_s - M_t} (q_t . k_s) v_s,        n_t . q_t likewise with n_0 and 1
//     S_C = e^{m_0 - M_C} S_0 + sum_s e^{a_s - M_C} k_s v_s^T,   n_C likewise,   m_C = F_C + M_C
// so no exponent is ever positive.  The gates alone fix M and m: one warp runs ahead with them.
//
// One CTA per (value tile of a head, sequence) walks the sequence.  TMEM: S1 = Q K^T, O1 = Q S_0, O2 = P V (128 columns each)
// and the state S^T (lane = value column) in fp32.  What enters the state or is read from it goes to the bf16 tensor cores
// as a hi + lo pair: S_0, the scaled keys e^{a_s - M_C} k_s, and the weights P.  Per chunk:
//     issuer    S1                O1            O2, S^T += V^T Kw
//     threads        Kw, n, decay     P, n . q                     outputs, S^T -> tile
// The keys are scaled in their TMA tile (hi; lo beside it); the P tiles overwrite the state tile, which is dead by then.
//
// A constant decay (kGated false; lightning attention) is the same with f = log decay, i = 0 and M_t = -F_t, so that m stays
// zero and the state is not rescaled: e^{a_s - M_t} = decay^{t - s}.  There is no normaliser and no q factor then.
#include "block_model.cuh"
#include "elem.cuh"
#include "mlstm.cuh"
#include "tc05.cuh"

namespace b200 {

namespace {
constexpr int kMC = 128;                                   // tokens per chunk
constexpr uint32_t kBlk = kMC * 128;                       // 128 rows of 64 bf16
constexpr uint32_t kMOffQ = 0, kMOffK = 2 * kBlk, kMOffV = 4 * kBlk, kMOffKlo = 6 * kBlk, kMOffA = 8 * kBlk;   // A: state tile hi | lo, then P hi | lo
constexpr uint32_t kMOffG = 12 * kBlk;                     // gate arrays, two buffers
constexpr uint32_t kGArr = 5 * kMC * 4 + 16;               // a2, M2, em, en, w, then keep
constexpr uint32_t kMOffN = kMOffG + 2 * ((kGArr + 127) / 128 * 128);   // n, two buffers
constexpr uint32_t kMOffR = kMOffN + 2 * kMC * 4;          // row sums of the two column halves
constexpr uint32_t kMOffBar = kMOffR + 2 * kMC * 4;
constexpr uint32_t kMSmem = kMOffBar + 256 + 1024;
constexpr int kMThreads = 320;                             // 8 compute warps, TMA + MMA issuer, gates
enum { M_FULL_QK = 0, M_FULL_V, M_S1, M_O1, M_ST, M_P, M_C3, M_GF, M_GE = M_GF + 2, M_BAR_COUNT = M_GE + 2 };
constexpr float kL2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2a(float x) {           // 2^x on the special-function unit; -inf -> 0
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void sync_compute() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
// 16-byte piece p (0..7) of row r in a 128-byte-swizzled tile
__device__ __forceinline__ uint32_t sw128(int r, int p) { return (uint32_t)(r * 128 + ((p ^ (r & 7)) << 4)); }
}  // namespace

// grid (heads * value tiles, sequences); ND = dp / 64 key blocks, NV = value blocks of a tile
template <int ND, int NV, bool kGated>
__global__ void __launch_bounds__(kMThreads, 1)
mlstm_chunk_kernel(const __grid_constant__ CUtensorMap map, const MlstmShape sh, const float* __restrict__ gates, int gate_pitch,
                   const float* __restrict__ bias, const LaSeqMeta* __restrict__ seqs, int max_seqs, float* __restrict__ state,
                   float* __restrict__ core, int* __restrict__ error_word) {
    extern __shared__ unsigned char smem_raw[];
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    unsigned char* sm = smem_raw + (base - raw);
    uint64_t* bars = reinterpret_cast<uint64_t*>(sm + kMOffBar);
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + M_BAR_COUNT);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    auto bar = [&](int i) { return base + kMOffBar + 8u * i; };

    const int h = blockIdx.x / sh.n_vt, tile = blockIdx.x % sh.n_vt;
    const LaSeqMeta sq = seqs[blockIdx.y];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int n_chunks = (sq.count + kMC - 1) / kMC;
    if (n_chunks <= 0 || sq.slot < 0 || sq.slot >= max_seqs) return;
    if (*reinterpret_cast<volatile int*>(error_word) != 0) return;   // an earlier CTA gave up: do not queue more bounded waits
    float* Sg = state + (size_t)sq.slot * sh.state_floats() + (size_t)blockIdx.x * sh.tile_floats();
    float* gn = Sg + (size_t)sh.dim * sh.vt;
    float* gm = gn + (sh.dim + 3) / 4 * 4;

    if (tid == 0) {
        for (int i = 0; i < M_BAR_COUNT; ++i) mbar_init(bar(i), (i == M_ST || i == M_P || i == M_GE || i == M_GE + 1) ? 256 : 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 8) {
        tmem_alloc(smem_u32(tmem_slot), 512);
        tmem_relinquish();
        if (lane == 0) tma_prefetch_desc(&map);
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot, tm_s1 = tmem, tm_o1 = tmem + 128, tm_o2 = tmem + 256, tm_st = tmem + 384;
    auto g_arr = [&](int b) { return reinterpret_cast<float*>(sm + kMOffG + b * ((kGArr + 127) / 128 * 128)); };

    if (warp == 8) {
        // ------------------------------ TMA + MMA issuer ------------------------------
        if (lane == 0) {
            constexpr uint32_t id_s1 = umma_idesc(kFmtBF16, 128, 128, 0, 0);
            constexpr uint32_t id_o1 = umma_idesc(kFmtBF16, 128, 64 * NV, 0, 0);
            constexpr uint32_t id_o2 = umma_idesc(kFmtBF16, 128, 64 * NV, 0, 1);
            constexpr uint32_t id_st = umma_idesc(kFmtBF16, 128, 64 * ND, 1, 1);
            const int xq = sh.off_q() + h * sh.dp, xk = sh.off_k() + h * sh.dp, xv = sh.off_v() + h * sh.vp + tile * kMlstmTile;
            auto load = [&](uint32_t off, int b, int x, int n, int c) {
                for (int i = 0; i < n; ++i) tma_load_2d(base + off + i * kBlk, &map, bar(b), x + 64 * i, sq.row0 + c * kMC);
            };
            mbar_arrive_expect_tx(bar(M_FULL_QK), 2 * ND * kBlk);
            load(kMOffQ, M_FULL_QK, xq, ND, 0);
            load(kMOffK, M_FULL_QK, xk, ND, 0);
            mbar_arrive_expect_tx(bar(M_FULL_V), NV * kBlk);
            load(kMOffV, M_FULL_V, xv, NV, 0);
            for (int c = 0; c < n_chunks; ++c) {
                const uint32_t par = c & 1;
                if (!mbar_wait(bar(M_FULL_QK), par, abort_flag)) break;
                tc_fence_after();
#pragma unroll
                for (int ks = 0; ks < 4 * ND; ++ks) {          // S1 = Q K^T
                    const uint32_t off = (ks >> 2) * kBlk + (ks & 3) * 32;
                    umma_f16(tm_s1, umma_smem_desc(base + kMOffQ + off, 16, 1024), umma_smem_desc(base + kMOffK + off, 16, 1024), id_s1, ks > 0);
                }
                umma_commit(bar(M_S1));
                if (!mbar_wait(bar(M_ST), par, abort_flag)) break;
                tc_fence_after();
#pragma unroll
                for (int hl = 0; hl < 2; ++hl)                 // O1 = Q S_0, state tile hi + lo
#pragma unroll
                    for (int ks = 0; ks < 4 * ND; ++ks) {
                        const uint32_t off = (ks >> 2) * kBlk + (ks & 3) * 32;
                        umma_f16(tm_o1, umma_smem_desc(base + kMOffQ + off, 16, 1024), umma_smem_desc(base + kMOffA + hl * 2 * kBlk + off, 16, 1024), id_o1,
                                 hl > 0 || ks > 0);
                    }
                umma_commit(bar(M_O1));
                if (!mbar_wait(bar(M_P), par, abort_flag)) break;
                tc_fence_after();
                if (c + 1 < n_chunks) {                        // nobody reads this chunk's Q any more
                    mbar_arrive_expect_tx(bar(M_FULL_QK), 2 * ND * kBlk);
                    load(kMOffQ, M_FULL_QK, xq, ND, c + 1);
                }
                if (!mbar_wait(bar(M_FULL_V), par, abort_flag)) break;
                tc_fence_after();
#pragma unroll
                for (int hl = 0; hl < 2; ++hl)
#pragma unroll
                    for (int ks = 0; ks < 8; ++ks) {           // O2 = P V;  S^T += V^T Kw
                        const uint64_t v = umma_smem_desc(base + kMOffV + ks * 2048, kBlk, 1024);
                        umma_f16(tm_o2, umma_smem_desc(base + kMOffA + hl * 2 * kBlk + (ks >> 2) * kBlk + (ks & 3) * 32, 16, 1024), v, id_o2, hl > 0 || ks > 0);
                        umma_f16(tm_st, v, umma_smem_desc(base + (hl ? kMOffKlo : kMOffK) + ks * 2048, kBlk, 1024), id_st, 1u);
                    }
                umma_commit(bar(M_C3));
                if (c + 1 < n_chunks) {
                    if (!mbar_wait(bar(M_C3), par, abort_flag)) break;
                    load(kMOffK, M_FULL_QK, xk, ND, c + 1);
                    mbar_arrive_expect_tx(bar(M_FULL_V), NV * kBlk);
                    load(kMOffV, M_FULL_V, xv, NV, c + 1);
                }
            }
        }
    } else if (warp == 9) {
        // ------------------------------ gates: four tokens per lane ------------------------------
        const float bi = bias[h], bf = bias[sh.heads + h], q_scale = 1.0f / sqrtf((float)sh.dim);
        float m0 = kGated ? *gm : 0.f;
        if constexpr (!kGated) {
            const float ld = bf;
            for (int c = 0; c < n_chunks; ++c) {
                const int b = c & 1, left = min(kMC, sq.count - c * kMC);
                if (c >= 2 && !mbar_wait_warp(bar(M_GE + b), ((c >> 1) - 1) & 1, abort_flag)) break;
                float* ga = g_arr(b);
                const float F_all = ld * (float)left;
                for (int t = lane; t < kMC; t += 32) {
                    const float F = ld * (float)min(t + 1, left);
                    ga[t] = t < left ? -F * kL2e : -INFINITY;
                    ga[kMC + t] = -F * kL2e;
                    ga[2 * kMC + t] = expf(F);
                    ga[4 * kMC + t] = t < left ? expf(ld * (float)(left - 1 - t)) : 0.f;
                }
                if (lane == 0) ga[5 * kMC] = expf(F_all);
                __syncwarp();
                if (lane == 0) mbar_arrive(bar(M_GF + b));
            }
        }
        if constexpr (kGated) for (int c = 0; c < n_chunks; ++c) {
            const int b = c & 1;
            float ig[4], F[4];
            float run = 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int t = c * kMC + 4 * lane + j;
                float f = 0.f;
                ig[j] = -INFINITY;
                if (t < sq.count) {
                    const float* g = gates + (size_t)(sq.row0 + t) * gate_pitch;
                    ig[j] = mlstm_log_input(g[h] + bi, sh.gate_cap);
                    f = mlstm_log_forget(g[sh.heads + h] + bf, sh.gate_cap);
                }
                run += f;
                F[j] = run;
            }
            float before = run;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, before, o);
                if (lane >= o) before += x;
            }
            const float F_all = __shfl_sync(0xffffffffu, before, 31);
            before -= run;
            float a[4], M[4], mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                F[j] += before;
                a[j] = ig[j] - F[j];
                mx = fmaxf(mx, a[j]);
                M[j] = mx;
            }
            float pm = mx;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, pm, o);
                if (lane >= o) pm = fmaxf(pm, x);
            }
            const float M_all = fmaxf(m0, __shfl_sync(0xffffffffu, pm, 31));
            float up = __shfl_up_sync(0xffffffffu, pm, 1);
            up = lane == 0 ? m0 : fmaxf(m0, up);
            if (c >= 2 && !mbar_wait_warp(bar(M_GE + b), ((c >> 1) - 1) & 1, abort_flag)) break;
            float* ga = g_arr(b);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int t = 4 * lane + j;
                const float Mt = fmaxf(up, M[j]);
                ga[t] = a[j] * kL2e;
                ga[kMC + t] = Mt * kL2e;
                ga[2 * kMC + t] = expf(m0 - Mt) * q_scale;
                ga[3 * kMC + t] = expf(-(F[j] + Mt));
                ga[4 * kMC + t] = expf(a[j] - M_all);
            }
            if (lane == 0) ga[5 * kMC] = expf(m0 - M_all);
            m0 = F_all + M_all;
            __syncwarp();
            if (lane == 0) mbar_arrive(bar(M_GF + b));
        }
        if (kGated && lane == 0 && !*abort_flag) *gm = m0;
    } else {
        // ------------------------------ compute warps ------------------------------
        const int r = tid & 127;     // TMEM lane: token of S1 / O1 / O2, value column of S^T
        const int hf = tid >> 7;     // which half of the columns
        const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
        const float q_scale = kGated ? 1.0f / sqrtf((float)sh.dim) : 1.0f;
        float* s_rs = reinterpret_cast<float*>(sm + kMOffR);
        auto s_n = [&](int b) { return reinterpret_cast<float*>(sm + kMOffN) + b * kMC; };
        bool ok = true;
        // S^T (TMEM) -> bf16 hi and lo tiles: row = value column, 32 key columns at a time
        auto state_cols = [&](int ch, const uint32_t (&sv)[32]) {
            if (r >= 64 * NV) return;
            unsigned char* t0 = sm + kMOffA + (ch >> 1) * kBlk;
#pragma unroll
            for (int q4 = 0; q4 < 4; ++q4) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    split_bf16x2(__uint_as_float(sv[q4 * 8 + 2 * e]), __uint_as_float(sv[q4 * 8 + 2 * e + 1]), hi[e], lo[e]);
                const uint32_t o = sw128(r, (ch & 1) * 4 + q4);
                *reinterpret_cast<uint4*>(t0 + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *reinterpret_cast<uint4*>(t0 + 2 * kBlk + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
        };
#pragma unroll 1
        for (int cc = 0; cc < ND; ++cc) {
            const int ch = hf * ND + cc;
            uint32_t sv[32];
#pragma unroll
            for (int e = 0; e < 32; ++e) {
                const int d = ch * 32 + e;
                sv[e] = (d < sh.dim && r < sh.vt) ? __float_as_uint(Sg[(size_t)d * sh.vt + r]) : 0u;
            }
            tmem_st32(tm_st + lane_base + ch * 32, sv);
            state_cols(ch, sv);
        }
        if (kGated && tid < kMC) s_n(0)[tid] = tid < sh.dim ? gn[tid] : 0.f;
        tmem_wait_st();
        fence_proxy_async_smem();
        tc_fence_before();
        mbar_arrive(bar(M_ST));
        sync_compute();
        for (int c = 0; c < n_chunks; ++c) {   // after a failed wait the warp keeps the barrier protocol going, without waiting or storing
            const uint32_t par = c & 1;
            const float* ga = g_arr(par);
            if (!mbar_wait_warp(bar(M_GF + par), (c >> 1) & 1, abort_flag)) ok = false;
            if (!mbar_wait_warp(bar(M_FULL_QK), par, abort_flag)) ok = false;
            const float keep = ga[5 * kMC];
            // n_0 . q of this thread's row, its half of the key columns
            float nq = 0.f;
            if constexpr (kGated) {
                const float* n0 = s_n(par);
#pragma unroll
                for (int p = 0; p < 4 * ND; ++p) {
                    const int oct = hf * 4 * ND + p;
                    const uint4 x = *reinterpret_cast<const uint4*>(sm + kMOffQ + (oct >> 3) * kBlk + sw128(r, oct & 7));
                    const float4 na = *reinterpret_cast<const float4*>(n0 + oct * 8), nb = *reinterpret_cast<const float4*>(n0 + oct * 8 + 4);
                    const float2 a = unpack_bf16x2(x.x), b = unpack_bf16x2(x.y), d = unpack_bf16x2(x.z), e = unpack_bf16x2(x.w);
                    nq += (a.x * na.x + a.y * na.y) + (b.x * na.z + b.y * na.w) + (d.x * nb.x + d.y * nb.y) + (e.x * nb.z + e.y * nb.w);
                }
                nq *= ga[2 * kMC + r];
            }
            // ---- keys times e^{a_s - M_C}: hi in place, lo beside it; their column sums advance n ----
            if (!mbar_wait_warp(bar(M_S1), par, abort_flag)) ok = false;
            tc_fence_after();
#pragma unroll 1
            for (int i = 0; i < ND; ++i) {
                const int oct = warp * ND + i;               // 8 ND octets of key columns, ND per warp
                unsigned char* t0 = sm + kMOffK + (oct >> 3) * kBlk;
                float cs[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int g = 0; g < 4; ++g) {
                    const int s = 32 * g + lane;
                    const float w = ga[4 * kMC + s];
                    uint4* p = reinterpret_cast<uint4*>(t0 + sw128(s, oct & 7));
                    const uint4 x = *p;
                    const uint32_t xs[4] = {x.x, x.y, x.z, x.w};
                    uint32_t hi[4], lo[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float2 v = unpack_bf16x2(xs[e]);
                        const float k0 = v.x * w, k1 = v.y * w;
                        cs[2 * e] += k0; cs[2 * e + 1] += k1;
                        split_bf16x2(k0, k1, hi[e], lo[e]);
                    }
                    *p = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                    *reinterpret_cast<uint4*>(reinterpret_cast<unsigned char*>(p) + (kMOffKlo - kMOffK)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
                }
                if constexpr (kGated) {
                    // eight sums over 32 lanes: halve the values while halving the lanes, lane groups of four end with one column each
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const bool top = lane & 16;
                        const float x = __shfl_xor_sync(0xffffffffu, top ? cs[e] : cs[e + 4], 16);
                        cs[e] = (top ? cs[e + 4] : cs[e]) + x;
                    }
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const bool top = lane & 8;
                        const float x = __shfl_xor_sync(0xffffffffu, top ? cs[e] : cs[e + 2], 8);
                        cs[e] = (top ? cs[e + 2] : cs[e]) + x;
                    }
                    {
                        const bool top = lane & 4;
                        const float x = __shfl_xor_sync(0xffffffffu, top ? cs[0] : cs[1], 4);
                        cs[0] = (top ? cs[1] : cs[0]) + x;
                    }
                    cs[0] += __shfl_xor_sync(0xffffffffu, cs[0], 2);
                    cs[0] += __shfl_xor_sync(0xffffffffu, cs[0], 1);
                    if ((lane & 3) == 0) {
                        const int d = oct * 8 + ((lane & 16) ? 4 : 0) + ((lane & 8) ? 2 : 0) + ((lane & 4) ? 1 : 0);
                        s_n(par ^ 1)[d] = keep * s_n(par)[d] + cs[0];
                    }
                }
            }
            // ---- the state decays to the chunk's end ----
#pragma unroll 1
            for (int cc = 0; cc < ND; ++cc) {
                const int ch = hf * ND + cc;
                uint32_t sv[32];
                tmem_ld32(tm_st + lane_base + ch * 32, sv);
                tmem_wait_ld();
#pragma unroll
                for (int e = 0; e < 32; ++e) sv[e] = __float_as_uint(__uint_as_float(sv[e]) * keep);
                tmem_st32(tm_st + lane_base + ch * 32, sv);
            }
            // ---- P = e^{a_s - M_t} (q_t . k_s) for s <= t, over the state tile ----
            if (!mbar_wait_warp(bar(M_O1), par, abort_flag)) ok = false;
            tc_fence_after();
            {
                const float Mt = ga[kMC + r];
                const bool none = hf == 1 && (warp & 3) < 2;          // rows 0 .. 63 see none of tokens 64 .. 127
#pragma unroll 1
                for (int cc = 0; cc < 2; ++cc) {
                    const int col0 = hf * 64 + cc * 32;
                    uint32_t s1[32];
                    if (!none) {
                        tmem_ld32(tm_s1 + lane_base + col0, s1);
                        tmem_wait_ld();
                    }
                    unsigned char* row = sm + kMOffA + hf * kBlk;
#pragma unroll
                    for (int q4 = 0; q4 < 4; ++q4) {
                        uint32_t hi[4] = {0u, 0u, 0u, 0u}, lo[4] = {0u, 0u, 0u, 0u};
                        if (!none) {
                            const float4 a0 = *reinterpret_cast<const float4*>(ga + col0 + q4 * 8), a1 = *reinterpret_cast<const float4*>(ga + col0 + q4 * 8 + 4);
                            const float as[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
                            float p[8];
#pragma unroll
                            for (int e = 0; e < 8; ++e) {
                                const int s = col0 + q4 * 8 + e;
                                p[e] = s <= r ? ex2a(as[e] - Mt) * (__uint_as_float(s1[q4 * 8 + e]) * q_scale) : 0.f;
                                nq += p[e];
                            }
#pragma unroll
                            for (int e = 0; e < 4; ++e) split_bf16x2(p[2 * e], p[2 * e + 1], hi[e], lo[e]);
                        }
                        const uint32_t o = sw128(r, cc * 4 + q4);
                        *reinterpret_cast<uint4*>(row + o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                        *reinterpret_cast<uint4*>(row + 2 * kBlk + o) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
                    }
                }
            }
            tmem_wait_st();
            fence_proxy_async_smem();
            tc_fence_before();
            mbar_arrive(bar(M_P));
            if constexpr (kGated) s_rs[hf * kMC + r] = nq;
            sync_compute();
            float inv = 1.0f;
            if constexpr (kGated) {
                nq += s_rs[(hf ^ 1) * kMC + r];
                inv = 1.0f / (fmaxf(fabsf(nq), ga[3 * kMC + r]) + 1e-6f);
            }
            const float em = ga[2 * kMC + r];
            mbar_arrive(bar(M_GE + par));
            // ---- outputs and the next state tile ----
            if (!mbar_wait_warp(bar(M_C3), par, abort_flag)) ok = false;
            tc_fence_after();
            float o[32 * NV];
#pragma unroll
            for (int cc = 0; cc < NV; ++cc) {
                const int ch = hf * NV + cc;
                uint32_t x1[32], x2[32];
                tmem_ld32(tm_o1 + lane_base + ch * 32, x1);
                tmem_ld32(tm_o2 + lane_base + ch * 32, x2);
                tmem_wait_ld();
#pragma unroll
                for (int e = 0; e < 32; ++e) o[cc * 32 + e] = (em * __uint_as_float(x1[e]) + __uint_as_float(x2[e])) * inv;
            }
            if (c + 1 < n_chunks) {
#pragma unroll 1
                for (int cc = 0; cc < ND; ++cc) {
                    const int ch = hf * ND + cc;
                    uint32_t sv[32];
                    tmem_ld32(tm_st + lane_base + ch * 32, sv);
                    tmem_wait_ld();
                    state_cols(ch, sv);
                }
                fence_proxy_async_smem();
                tc_fence_before();
                mbar_arrive(bar(M_ST));
            }
            const int t = c * kMC + r;
            if (ok && t < sq.count) {
                float* dst = core + (size_t)(sq.row0 + t) * (sh.heads * sh.vp) + h * sh.vp + tile * kMlstmTile + hf * 32 * NV;
#pragma unroll
                for (int e = 0; e < 8 * NV; ++e)
                    if (tile * kMlstmTile + hf * 32 * NV + 4 * e < sh.vp)
                        *reinterpret_cast<float4*>(dst + 4 * e) = make_float4(o[4 * e], o[4 * e + 1], o[4 * e + 2], o[4 * e + 3]);
            }
        }
        // ---- final state ----
        if (ok) {
#pragma unroll 1
            for (int cc = 0; cc < ND; ++cc) {
                const int ch = hf * ND + cc;
                uint32_t sv[32];
                tmem_ld32(tm_st + lane_base + ch * 32, sv);
                tmem_wait_ld();
#pragma unroll
                for (int e = 0; e < 32; ++e) {
                    const int d = ch * 32 + e;
                    if (d < sh.dim && r < sh.vt) Sg[(size_t)d * sh.vt + r] = __uint_as_float(sv[e]);
                }
            }
            if (kGated && tid < sh.dim) gn[tid] = s_n(n_chunks & 1)[tid];
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 8) {
        tc_fence_after();
        tmem_dealloc(tmem, 512);
    }
    if (tid == 0 && *abort_flag) atomicExch(error_word, 9);
}

bool mlstm_chunk_fits(const MlstmShape& sh) { return sh.dp <= 128; }

// qkvg: bf16 [rows][cols]; gates: fp32 [rows][gate_pitch], input then forget pre-activations (not gated: unused, bias holds decays and log decays).
int launch_mlstm_chunk(const MlstmShape& sh, const void* qkvg, int rows, const float* gates, int gate_pitch, const float* bias,
                       const LaSeqMeta* d_seqs, int n_seqs, int max_seqs, float* state, float* core, int* d_error, cudaStream_t s) {
    CUtensorMap map;
    const uint64_t dims[2] = {(uint64_t)sh.cols(), (uint64_t)rows};
    const uint64_t str[1] = {(uint64_t)sh.cols() * 2};
    const uint32_t box[2] = {64, (uint32_t)kMC};
    B2_TRY(make_tensor_map(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, qkvg, dims, str, box));
    static PerDeviceOnce once;
    B2_PER_DEVICE_ONCE(once,
        for (auto k : {mlstm_chunk_kernel<1, 1, true>, mlstm_chunk_kernel<1, 2, true>, mlstm_chunk_kernel<2, 1, true>, mlstm_chunk_kernel<2, 2, true>,
                       mlstm_chunk_kernel<1, 1, false>, mlstm_chunk_kernel<1, 2, false>, mlstm_chunk_kernel<2, 1, false>, mlstm_chunk_kernel<2, 2, false>})
            B2_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, kMSmem)));
    const dim3 grid(sh.heads * sh.n_vt, n_seqs);
    auto go = [&](auto kernel) { kernel<<<grid, kMThreads, kMSmem, s>>>(map, sh, gates, gate_pitch, bias, d_seqs, max_seqs, state, core, d_error); };
    const bool d2 = sh.dp > 64, v2 = sh.vp > 64;
    auto pick = [&](auto gated) {
        constexpr bool kGated = decltype(gated)::value;
        if (d2 && v2) go(mlstm_chunk_kernel<2, 2, kGated>);
        else if (d2) go(mlstm_chunk_kernel<2, 1, kGated>);
        else if (v2) go(mlstm_chunk_kernel<1, 2, kGated>);
        else go(mlstm_chunk_kernel<1, 1, kGated>);
    };
    if (sh.gated) pick(std::true_type{}); else pick(std::false_type{});
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
