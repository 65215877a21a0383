// Differential flash attention for prefill on tcgen05, keys and values straight from the cache pages (bf16).
//
// Persistent CTAs walk (128-query tile, head) items.  Per 64-key page: S_m = Q_m K_m^T for both maps m, then O_m += P_m V over the
// same values.  Each of the two softmax warpgroups owns a map, one thread per query row with all 64 scores of a page, so the
// running maximum and sum need no exchange; both accumulators live in TMEM and meet in the epilogue, where every thread of a row
// takes half of the value columns: o = a1 - lambda a2, over its root mean square, times 1 - diff.
// The keys of an item are the pages that hold kept positions, then the pages its window touches; a page is one TMA box per 64
// columns.  S is double-buffered per map (4 x 64 TMEM columns), O takes up to 2 x 128.  All waits are bounded.
#include "block_model.cuh"
#include "elem.cuh"
#include "tc05.cuh"

#include <algorithm>

namespace b200 {

namespace {
constexpr int kDM = 128, kDN = 64, kDThreads = 320;
constexpr uint32_t kDQBlk = kDM * 128, kDKBlk = kDN * 128, kDPBuf = kDM * 128;
static_assert(kDN == kPageTokens, "a key tile is a cache page");
// S, P barriers: index + 2 * map + buffer
enum { D_Q = 0, D_QE, D_KF, D_KE = D_KF + 3, D_VF = D_KE + 3, D_VE = D_VF + 3, D_SF = D_VE + 3, D_SE = D_SF + 4, D_PF = D_SE + 4, D_PV = D_PF + 4, D_OF = D_PV + 4,
       D_OD, D_BARS };
struct DpShape {
    int heads, kv_heads, per, nd, nv, vdim, window, keep;   // nd, nv: blocks of 64 columns of a map, of the values
    float sc, lambda, out_scale, eps;                       // sc: score factor times log2 e
    uint32_t off_k, off_v, off_p, off_bar;
};
__device__ __forceinline__ float ex2d(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
}  // namespace

template <int NST>
__global__ void __launch_bounds__(kDThreads, 1)
diff_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv, const __grid_constant__ CUtensorMap map_o,
                    const DpShape L, const int* __restrict__ block_table, int max_pages, const DiffTile* __restrict__ tiles, int n_items,
                    __nv_bfloat16* __restrict__ out, int* __restrict__ error_word) {
    extern __shared__ __align__(1024) unsigned char sm[];
    const uint32_t base = smem_u32(sm);
    if (base & 1023u) {            // the 128-byte swizzle needs 1024-byte aligned tiles
        if (threadIdx.x == 0) atomicExch(error_word, 8);
        return;
    }
    uint64_t* bars = reinterpret_cast<uint64_t*>(sm + L.off_bar);
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + D_BARS);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    float* x_l = reinterpret_cast<float*>(sm + L.off_bar + 512);       // row sums of the two maps, then sums of squares of the two column halves
    auto bar = [&](int i) { return base + L.off_bar + 8u * i; };
    if (*reinterpret_cast<volatile int*>(error_word) != 0) return;     // an earlier launch gave up: do not queue more bounded waits
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int cta = blockIdx.x, n_cta = gridDim.x;
    const int n_my = (cta < n_items) ? (n_items - cta + n_cta - 1) / n_cta : 0;
    struct Item { DiffTile t; int head, kept, w0, n_kt; };             // pages of kept positions, first page behind them, pages in all
    auto item = [&](int i) -> Item {
        const int w = cta + i * n_cta;
        Item x;
        x.t = tiles[w / L.heads];
        x.head = w % L.heads;
        const int end = x.t.q_pos0 + x.t.n_rows, first = L.window > 0 ? max(0, x.t.q_pos0 - L.window + 1) : 0;
        x.kept = (min(L.keep, end) + kDN - 1) / kDN;
        x.w0 = max(x.kept, first / kDN);
        x.n_kt = x.kept + max(0, (end - 1) / kDN - x.w0 + 1);
        return x;
    };
    auto page_of = [](const Item& x, int j) { return j < x.kept ? j : x.w0 + j - x.kept; };

    if (threadIdx.x == 0) {
        for (int i = 0; i < D_BARS; ++i)
            mbar_init(bar(i), i == D_OD ? 256 : ((i >= D_SE && i < D_SE + 4) || (i >= D_PF && i < D_PF + 4)) ? 128 : 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 9) {
        tmem_alloc(smem_u32(tmem_slot), 512);
        tmem_relinquish();
    }
    if (warp == 8 && lane == 0) { tma_prefetch_desc(&map_q); tma_prefetch_desc(&map_kv); tma_prefetch_desc(&map_o); }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot, tmem_o = tmem + 256;             // S of map m, buffer b at (2 m + b) * 64; O of map m at m * 64 nv

    if (warp == 8) {
        // ------------------------------ TMA producer: Q, K and V advance independently ------------------------------
        if (lane == 0) {
            const int nq = 2 * L.nd;
            int iq = 0, ik = 0, jk = 0, gk = 0, iv = 0, jv = 0, gv = 0, rk = 0, rv = 0;
            Item tk = {}, tv = {};
            auto row_of = [&](const Item& x, int j) {                  // first cache row of the item's j-th page
                return (block_table[(size_t)x.t.slot * max_pages + page_of(x, j)] * L.kv_heads + x.head / L.per) * kDN;
            };
            if (n_my > 0) { tk = item(0); tv = tk; rk = rv = row_of(tk, 0); }
            const uint64_t t0 = global_timer_ns();
            uint32_t idle = 0;
            while (iq < n_my || ik < n_my || iv < n_my) {
                bool progressed = false;
                if (iq < n_my && (iq == 0 || mbar_test_wait(bar(D_QE), (iq - 1) & 1))) {
                    const Item tq = item(iq);
                    mbar_arrive_expect_tx(bar(D_Q), nq * kDQBlk);
                    for (int b = 0; b < nq; ++b) tma_load_2d(base + b * kDQBlk, &map_q, bar(D_Q), (tq.head * nq + b) * 64, tq.t.q_row0);
                    ++iq;
                    progressed = true;
                }
                if (ik < n_my && (gk < NST || mbar_test_wait(bar(D_KE + gk % NST), (gk / NST - 1) & 1))) {
                    const int s = gk % NST;
                    const uint32_t dst = base + L.off_k + s * nq * kDKBlk;
                    mbar_arrive_expect_tx(bar(D_KF + s), nq * kDKBlk);
                    for (int b = 0; b < nq; ++b) tma_load_2d(dst + b * kDKBlk, &map_kv, bar(D_KF + s), b * 64, rk);
                    ++gk;
                    if (++jk == tk.n_kt) { jk = 0; if (++ik < n_my) tk = item(ik); }
                    if (ik < n_my) rk = row_of(tk, jk);
                    progressed = true;
                }
                if (iv < n_my && (gv < NST || mbar_test_wait(bar(D_VE + gv % NST), (gv / NST - 1) & 1))) {
                    const int s = gv % NST;
                    mbar_arrive_expect_tx(bar(D_VF + s), L.nv * kDKBlk);
                    for (int b = 0; b < L.nv; ++b) tma_load_2d(base + L.off_v + (s * L.nv + b) * kDKBlk, &map_kv, bar(D_VF + s), (nq + b) * 64, rv);
                    ++gv;
                    if (++jv == tv.n_kt) { jv = 0; if (++iv < n_my) tv = item(iv); }
                    if (iv < n_my) rv = row_of(tv, jv);
                    progressed = true;
                }
                if (!progressed && ((++idle & 255u) == 0u)) {
                    if (*abort_flag) break;
                    if (global_timer_ns() - t0 > 4000000000ull) { *abort_flag = 1; break; }
                }
            }
        }
    } else if (warp == 9) {
        // ------------------------------ MMA issuer ------------------------------
        if (lane == 0) {
            constexpr uint32_t id_s = umma_idesc(kFmtBF16, kDM, kDN, 0, 0);
            const uint32_t id_pv = umma_idesc(kFmtBF16, kDM, 64 * L.nv, 0, 1);
            // PV products of global step g; `first` overwrites O (the previous item's epilogue has read it), after `last` O is final
            auto issue_pv = [&](int g, bool first, bool last, int it) -> bool {
                const int b = g & 1, s = g % NST;
                if (!mbar_wait(bar(D_VF + s), (g / NST) & 1, abort_flag)) return false;
                if (first && it > 0 && !mbar_wait(bar(D_OD), (it - 1) & 1, abort_flag)) return false;
                for (int m = 0; m < 2; ++m) {
                    if (!mbar_wait(bar(D_PF + 2 * m + b), (g >> 1) & 1, abort_flag)) return false;
                    tc_fence_after();
#pragma unroll
                    for (int ks = 0; ks < 4; ++ks)
                        umma_f16(tmem_o + m * 64 * L.nv, umma_smem_desc(base + L.off_p + (2 * m + b) * kDPBuf + ks * 32, 16, 1024),
                                 umma_smem_desc(base + L.off_v + s * L.nv * kDKBlk + ks * 2048, kDKBlk, 1024), id_pv, (!first || ks > 0) ? 1u : 0u);
                    umma_commit(bar(D_PV + 2 * m + b));
                }
                umma_commit(bar(D_VE + s));
                if (last) umma_commit(bar(D_OF));
                return true;
            };
            bool ok = true, pending = false, pfirst = false, plast = false;
            int pg = 0, pitem = 0, gs = 0;
            for (int i = 0; ok && i < n_my; ++i) {
                const int n_kt = item(i).n_kt;
                if (pending) {         // the previous item's last PV goes out before the wait for this item's Q tile
                    if (!issue_pv(pg, pfirst, plast, pitem)) { ok = false; break; }
                    pending = false;
                }
                if (!mbar_wait(bar(D_Q), i & 1, abort_flag)) { ok = false; break; }
                for (int j = 0; ok && j < n_kt; ++j, ++gs) {
                    const int b = gs & 1, s = gs % NST;
                    if (!mbar_wait(bar(D_KF + s), (gs / NST) & 1, abort_flag)) { ok = false; break; }
                    for (int m = 0; m < 2; ++m) {
                        if (gs >= 2 && !mbar_wait(bar(D_SE + 2 * m + b), ((gs >> 1) - 1) & 1, abort_flag)) { ok = false; break; }
                        tc_fence_after();
                        for (int blk = 0; blk < L.nd; ++blk)
#pragma unroll
                            for (int ks = 0; ks < 4; ++ks)
                                umma_f16(tmem + (2 * m + b) * kDN, umma_smem_desc(base + (m * L.nd + blk) * kDQBlk + ks * 32, 16, 1024),
                                         umma_smem_desc(base + L.off_k + ((s * 2 + m) * L.nd + blk) * kDKBlk + ks * 32, 16, 1024), id_s, (blk > 0 || ks > 0) ? 1u : 0u);
                        umma_commit(bar(D_SF + 2 * m + b));
                    }
                    if (!ok) break;
                    umma_commit(bar(D_KE + s));
                    if (j == n_kt - 1) umma_commit(bar(D_QE));
                    if (pending && !issue_pv(pg, pfirst, plast, pitem)) { ok = false; break; }
                    pending = true; pg = gs; pfirst = (j == 0); plast = (j == n_kt - 1); pitem = i;
                }
            }
            if (ok && pending) issue_pv(pg, pfirst, plast, pitem);
        }
    } else {
        // ------------------------------ softmax / correction / epilogue ------------------------------
        const int r = threadIdx.x & 127;                 // query row == TMEM lane
        const int m = threadIdx.x >> 7;                  // map of this thread / which half of each 64 output columns
        const int wrow = (warp & 3) * 32;
        const uint32_t lane_base = (uint32_t)wrow << 16;
        const int pair_bar = 1 + (warp & 3);             // named barrier shared by the two warps that cover the same rows
        const int W = L.window > 0 ? L.window : 1 << 30;
        const uint32_t tm_s = tmem + 2 * m * kDN + lane_base, tm_o = tmem_o + m * 64 * L.nv + lane_base;
        const float sc = L.sc;
        bool ok = true;
        int gs = 0;
        for (int it = 0; it < n_my; ++it) {
            const Item im = item(it);
            const int q_pos = im.t.q_pos0 + r, w_lo = im.t.q_pos0 + wrow;     // this row's position, the warp's first
            float m_ref = -INFINITY, l = 0.f;
            for (int j = 0; j < im.n_kt; ++j, ++gs) {
                const int b = gs & 1;
                if (!mbar_wait_warp(bar(D_SF + 2 * m + b), (gs >> 1) & 1, abort_flag)) ok = false;
                tc_fence_after();
                uint32_t s0[32], s1[32];
                tmem_ld32(tm_s + b * kDN, s0);
                tmem_ld32(tm_s + b * kDN + 32, s1);
                tmem_wait_ld();
                tc_fence_before();
                mbar_arrive(bar(D_SE + 2 * m + b));
                const int kp0 = page_of(im, j) * kDN;
                float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
                if (kp0 + kDN - 1 > w_lo || (kp0 <= w_lo + 31 - W && kp0 + kDN > L.keep)) {     // warp-uniform: an edge may cross this page
                    const int hi = q_pos - kp0, lo = hi - W, kc = L.keep - kp0;                 // visible: c <= hi and (c > lo or c < kc)
#pragma unroll
                    for (int c = 0; c < 32; ++c) {
                        const float v0 = (c <= hi && (c > lo || c < kc)) ? __uint_as_float(s0[c]) : -INFINITY;
                        const float v1 = (c + 32 <= hi && (c + 32 > lo || c + 32 < kc)) ? __uint_as_float(s1[c]) : -INFINITY;
                        s0[c] = __float_as_uint(v0);
                        s1[c] = __float_as_uint(v1);
                        mx4[c & 3] = fmaxf(mx4[c & 3], fmaxf(v0, v1));
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < 32; ++c) mx4[c & 3] = fmaxf(mx4[c & 3], fmaxf(__uint_as_float(s0[c]), __uint_as_float(s1[c])));
                }
                const float m_new = fmaxf(m_ref, fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * sc);      // -inf while the row has seen no key
                const bool need = (m_new - m_ref > 8.0f);        // true at the row's first key (m_ref = -inf)
                if (__any_sync(0xffffffffu, need)) {
                    if (j > 0) {
                        if (!mbar_wait_warp(bar(D_PV + 2 * m + ((gs - 1) & 1)), ((gs - 1) >> 1) & 1, abort_flag)) ok = false;
                        tc_fence_after();
                        const float alpha = m_new == m_ref ? 1.0f : exp2f(m_ref - m_new);
                        l *= alpha;
#pragma unroll 1
                        for (int cc = 0; cc < 2 * L.nv; ++cc) {
                            uint32_t o[32];
                            tmem_ld32(tm_o + cc * 32, o);
                            tmem_wait_ld();
#pragma unroll
                            for (int c = 0; c < 32; ++c) o[c] = __float_as_uint(__uint_as_float(o[c]) * alpha);
                            tmem_st32(tm_o + cc * 32, o);
                        }
                        tmem_wait_st();
                    }
                    m_ref = m_new;
                }
                // P = 2^(s * scale - m_ref) as bf16 into the swizzled K-major A tile
                if (gs >= 2 && !mbar_wait_warp(bar(D_PV + 2 * m + b), ((gs >> 1) - 1) & 1, abort_flag)) ok = false;
                const float m_use = m_ref == -INFINITY ? 0.f : m_ref;
                unsigned char* prow = sm + L.off_p + (2 * m + b) * kDPBuf + r * 128;
                float ls4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int c8 = 0; c8 < 8; ++c8) {
                    uint32_t pk[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int c = (c8 & 3) * 8 + 2 * e;
                        const float x0 = __uint_as_float(c8 < 4 ? s0[c] : s1[c]), x1 = __uint_as_float(c8 < 4 ? s0[c + 1] : s1[c + 1]);
                        const float p0 = ex2d(fmaf(x0, sc, -m_use)), p1 = ex2d(fmaf(x1, sc, -m_use));
                        ls4[e] += p0 + p1;
                        pk[e] = pack_bf16x2(p0, p1);
                    }
                    *reinterpret_cast<uint4*>(prow + ((c8 ^ (r & 7)) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                }
                l += (ls4[0] + ls4[1]) + (ls4[2] + ls4[3]);
                fence_proxy_async_smem();
                tc_fence_before();
                mbar_arrive(bar(D_PF + 2 * m + b));
            }
            // ---- both maps meet: this thread takes its half of every 64 value columns ----
            x_l[m * 128 + r] = l;
            asm volatile("bar.sync %0, 64;" ::"r"(pair_bar) : "memory");
            const float i1 = 1.0f / x_l[r], i2 = L.lambda / x_l[128 + r];
            if (!mbar_wait_warp(bar(D_OF), it & 1, abort_flag)) ok = false;
            tc_fence_after();
            uint32_t d[2][32];
            float ss = 0.f;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                if (k >= L.nv) break;
                uint32_t o2[32];
                tmem_ld32(tmem_o + lane_base + (2 * k + m) * 32, d[k]);
                tmem_ld32(tmem_o + lane_base + (2 * (L.nv + k) + m) * 32, o2);
                tmem_wait_ld();
#pragma unroll
                for (int c = 0; c < 32; ++c) {
                    const float x = __uint_as_float(d[k][c]) * i1 - __uint_as_float(o2[c]) * i2;
                    d[k][c] = __float_as_uint(x);
                    ss += x * x;
                }
            }
            tc_fence_before();
            mbar_arrive(bar(D_OD));            // this thread has read its part of O: the next item's first PV may overwrite it
            x_l[256 + m * 128 + r] = ss;
            asm volatile("bar.sync %0, 64;" ::"r"(pair_bar) : "memory");
            ss += x_l[256 + (m ^ 1) * 128 + r];
            const float f = L.out_scale / sqrtf(ss / (float)L.vdim + L.eps);
            // full tiles through shared memory (the idle P buffers) and tiled TMA stores, others from registers
            const bool via_tma = im.t.n_rows == kDM;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                if (k >= L.nv) break;
                unsigned char* srow = sm + L.off_p + k * kDPBuf + r * 128;
                __nv_bfloat16* dst = out + (size_t)(im.t.q_row0 + r) * L.heads * L.nv * 64 + (im.head * L.nv + k) * 64 + m * 32;
#pragma unroll
                for (int q8 = 0; q8 < 4; ++q8) {
                    uint32_t h[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) h[e] = pack_bf16x2(__uint_as_float(d[k][8 * q8 + 2 * e]) * f, __uint_as_float(d[k][8 * q8 + 2 * e + 1]) * f);
                    if (via_tma) *reinterpret_cast<uint4*>(srow + (((m * 4 + q8) ^ (r & 7)) << 4)) = make_uint4(h[0], h[1], h[2], h[3]);
                    else if (r < im.t.n_rows && ok) *reinterpret_cast<uint4*>(dst + 8 * q8) = make_uint4(h[0], h[1], h[2], h[3]);
                }
            }
            if (via_tma) {
                fence_proxy_async_smem();
                asm volatile("bar.sync 5, 256;" ::: "memory");
                if (threadIdx.x == 0) {
                    if (ok)
                        for (int k = 0; k < L.nv; ++k) tma_store_2d(&map_o, base + L.off_p + k * kDPBuf, (im.head * L.nv + k) * 64, im.t.q_row0);
                    bulk_commit_group();
                    bulk_wait_group_read0();
                }
                asm volatile("bar.sync 5, 256;" ::: "memory");     // the P buffers go back to the softmax of the next item
            }
        }
    }
    if (threadIdx.x == 0) bulk_wait_group0();          // this thread's TMA stores have reached global memory
    tc_fence_before();
    __syncthreads();
    if (warp == 9) {
        tc_fence_after();
        tmem_dealloc(tmem, 512);
    }
    if (threadIdx.x == 0 && *abort_flag) atomicExch(error_word, 5);
}

static uint32_t dp_smem(int nd, int nv, int stages) { return 2 * nd * kDQBlk + stages * (2 * nd + nv) * kDKBlk + 4 * kDPBuf + 512 + 2048; }

bool diff_prefill_fits(const DiffShape& sh) {
    return sh.dp % 64 == 0 && sh.vp % 64 == 0 && sh.dp <= 128 && sh.vp <= 128 && sh.scale > 0.f && dp_smem(sh.dp / 64, sh.vp / 64, 2) <= 227 * 1024;
}

// q [rows][heads][2][dp], out [rows][heads][vp], bf16.
int launch_diff_prefill(const DiffShape& sh, float lambda, const void* q, int rows, const LatentView& cache, const DiffTile* d_tiles, int n_tiles,
                        void* out, int* d_error, cudaStream_t s) {
    if (n_tiles <= 0) return 0;
    auto map = [&](CUtensorMap* m, const void* p, int cols, uint64_t pitch, uint64_t n, int box_rows) -> int {
        const uint64_t dims[2] = {(uint64_t)cols, n};
        const uint64_t str[1] = {pitch * 2};
        const uint32_t box[2] = {64, (uint32_t)box_rows};
        return make_tensor_map(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p, dims, str, box);
    };
    CUtensorMap mq, mkv, mo;
    B2_TRY(map(&mq, q, sh.q_cols(), sh.q_cols(), rows, kDM));
    B2_TRY(map(&mkv, cache.rows, 2 * sh.dp + sh.vp, sh.hp(), (uint64_t)cache.num_pages * sh.kv_heads * kPageTokens, kDN));
    B2_TRY(map(&mo, out, sh.heads * sh.vp, (uint64_t)sh.heads * sh.vp, rows, kDM));
    static PerDeviceOnce once;
    B2_PER_DEVICE_ONCE(once,
        B2_CUDA(cudaFuncSetAttribute(diff_prefill_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        B2_CUDA(cudaFuncSetAttribute(diff_prefill_kernel<3>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024)));
    int n_sm = 0;
    B2_TRY(device_sm_count(&n_sm));
    const int nd = sh.dp / 64, nv = sh.vp / 64, stages = dp_smem(nd, nv, 3) <= 227 * 1024 ? 3 : 2, n_items = n_tiles * sh.heads;
    DpShape L{sh.heads, sh.kv_heads, sh.heads / sh.kv_heads, nd, nv, sh.vdim, sh.window, sh.keep, sh.scale * 1.4426950408889634f, lambda, 1.0f - sh.diff, sh.eps};
    L.off_k = 2 * nd * kDQBlk;
    L.off_v = L.off_k + stages * 2 * nd * kDKBlk;
    L.off_p = L.off_v + stages * nv * kDKBlk;
    L.off_bar = L.off_p + 4 * kDPBuf;
    auto go = [&](auto kernel) {
        kernel<<<std::min(n_items, n_sm), kDThreads, dp_smem(nd, nv, stages), s>>>(mq, mkv, mo, L, cache.block_table, cache.max_pages_per_seq, d_tiles, n_items,
                                                                                   (__nv_bfloat16*)out, d_error);
    };
    if (stages == 3) go(diff_prefill_kernel<3>); else go(diff_prefill_kernel<2>);
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
