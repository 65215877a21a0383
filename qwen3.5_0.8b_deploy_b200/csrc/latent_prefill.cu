// Sliding-window flash attention for prefill on tcgen05, with keys and values up-projected from staged latents (bf16).
//
// The schedule of the causal prefill kernel (fa_prefill.cu): persistent CTAs walk (128-query tile, head) items, eight softmax
// warps (two threads per query row), a TMA lane and an MMA lane, S double-buffered in TMEM, O in TMEM, all ring barriers on
// step counters that run across items.  What differs: a key is [unrotated part of the head | rotated part shared by all
// heads], fetched from two tensors; sizes come in blocks of 64 columns (query / key blocks <= 4, value blocks <= 4), with a
// third K / V stage where shared memory allows; and a tile's key range starts where the window of its first query does, so
// a row may see nothing of its first key tiles.
#include "block_model.cuh"
#include "elem.cuh"
#include "tc05.cuh"

#include <algorithm>

namespace b200 {

namespace {
constexpr int kLM = 128, kLN = 64, kLThreads = 320;
constexpr uint32_t kQBlk = kLM * 128, kKBlk = kLN * 128, kPBuf = kLM * 128;
enum { L_Q = 0, L_QE = 1, L_KF = 2, L_KE = 5, L_VF = 8, L_VE = 11, L_SF = 14, L_SE = 16, L_PF = 18, L_PV = 20, L_OF = 22, L_OD = 23, L_BARS = 24 };
struct LpShape {
    int heads, nd, nr, nv, window;     // blocks of 64 columns: unrotated, rotated, value
    float sc;                          // score scale times log2 e
    uint32_t off_k, off_v, off_p, off_bar;
};
__device__ __forceinline__ float ex2p(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
}  // namespace

template <int NST>
__global__ void __launch_bounds__(kLThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_r,
                      const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_o, const LpShape L,
                      const LatentTile* __restrict__ tiles, int n_items, __nv_bfloat16* __restrict__ out, int* __restrict__ error_word) {
    extern __shared__ __align__(1024) unsigned char sm[];
    const uint32_t base = smem_u32(sm);
    if (base & 1023u) {            // the 128-byte swizzle needs 1024-byte aligned tiles
        if (threadIdx.x == 0) atomicExch(error_word, 8);
        return;
    }
    uint64_t* bars = reinterpret_cast<uint64_t*>(sm + L.off_bar);
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + L_BARS);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    float* x_mx = reinterpret_cast<float*>(sm + L.off_bar + 256);      // row-maximum exchange [2 tiles][2 halves][128]
    auto bar = [&](int i) { return base + L.off_bar + 8u * i; };
    if (*reinterpret_cast<volatile int*>(error_word) != 0) return;     // an earlier launch gave up: do not queue more bounded waits
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int cta = blockIdx.x, n_cta = gridDim.x;
    const int n_my = (cta < n_items) ? (n_items - cta + n_cta - 1) / n_cta : 0;
    const int nq = L.nd + L.nr;
    struct Item { LatentTile t; int head, key0, row0, n_kt; };        // key0: first position of the first key tile, row0: its staging row
    auto item = [&](int i) -> Item {
        const int w = cta + i * n_cta;
        Item x;
        x.t = tiles[w / L.heads];
        x.head = w % L.heads;
        x.key0 = max(x.t.ctx_pos0, L.window > 0 ? x.t.q_pos0 - L.window + 1 : 0);
        x.row0 = x.t.ctx_row0 + (x.key0 - x.t.ctx_pos0);
        x.n_kt = (x.t.q_pos0 + x.t.n_rows - x.key0 + kLN - 1) / kLN;
        return x;
    };

    if (threadIdx.x == 0) {
        for (int i = 0; i < L_BARS; ++i) {
            const bool many = (i == L_SE || i == L_SE + 1 || i == L_PF || i == L_PF + 1 || i == L_OD);
            mbar_init(bar(i), many ? 256 : 1);
        }
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 9) {
        tmem_alloc(smem_u32(tmem_slot), 512);
        tmem_relinquish();
    }
    if (warp == 8 && lane == 0) {
        tma_prefetch_desc(&map_q); tma_prefetch_desc(&map_k); tma_prefetch_desc(&map_r); tma_prefetch_desc(&map_v); tma_prefetch_desc(&map_o);
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot, tmem_o = tmem + 128;

    if (warp == 8) {
        // ------------------------------ TMA producer: Q, K and V advance independently ------------------------------
        if (lane == 0) {
            int iq = 0, ik = 0, jk = 0, gk = 0, iv = 0, jv = 0, gv = 0;
            Item tk = {}, tv = {};
            if (n_my > 0) { tk = item(0); tv = tk; }
            const uint64_t t0 = global_timer_ns();
            uint32_t idle = 0;
            while (iq < n_my || ik < n_my || iv < n_my) {
                bool progressed = false;
                if (iq < n_my && (iq == 0 || mbar_test_wait(bar(L_QE), (iq - 1) & 1))) {
                    const Item tq = item(iq);
                    mbar_arrive_expect_tx(bar(L_Q), nq * kQBlk);
                    for (int b = 0; b < nq; ++b) tma_load_2d(base + b * kQBlk, &map_q, bar(L_Q), (tq.head * nq + b) * 64, tq.t.q_row0);
                    ++iq;
                    progressed = true;
                }
                if (ik < n_my && (gk < NST || mbar_test_wait(bar(L_KE + gk % NST), (gk / NST - 1) & 1))) {
                    const int s = gk % NST, row = tk.row0 + jk * kLN;
                    const uint32_t dst = base + L.off_k + s * nq * kKBlk;
                    mbar_arrive_expect_tx(bar(L_KF + s), nq * kKBlk);
                    for (int b = 0; b < L.nd; ++b) tma_load_2d(dst + b * kKBlk, &map_k, bar(L_KF + s), (tk.head * L.nd + b) * 64, row);
                    for (int b = 0; b < L.nr; ++b) tma_load_2d(dst + (L.nd + b) * kKBlk, &map_r, bar(L_KF + s), b * 64, row);
                    ++gk;
                    if (++jk == tk.n_kt) { jk = 0; if (++ik < n_my) tk = item(ik); }
                    progressed = true;
                }
                if (iv < n_my && (gv < NST || mbar_test_wait(bar(L_VE + gv % NST), (gv / NST - 1) & 1))) {
                    const int s = gv % NST, row = tv.row0 + jv * kLN;
                    mbar_arrive_expect_tx(bar(L_VF + s), L.nv * kKBlk);
                    for (int b = 0; b < L.nv; ++b)
                        tma_load_2d(base + L.off_v + (s * L.nv + b) * kKBlk, &map_v, bar(L_VF + s), (tv.head * L.nv + b) * 64, row);
                    ++gv;
                    if (++jv == tv.n_kt) { jv = 0; if (++iv < n_my) tv = item(iv); }
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
            constexpr uint32_t id_s = umma_idesc(kFmtBF16, kLM, kLN, 0, 0);
            const uint32_t id_pv = umma_idesc(kFmtBF16, kLM, 64 * L.nv, 0, 1);
            // PV product of global step g; `first` overwrites O (the previous item's epilogue has read it), after `last` O is final
            auto issue_pv = [&](int g, bool first, bool last, int it) -> bool {
                const int b = g & 1, s = g % NST;
                if (!mbar_wait(bar(L_VF + s), (g / NST) & 1, abort_flag)) return false;
                if (!mbar_wait(bar(L_PF + b), (g >> 1) & 1, abort_flag)) return false;
                if (first && it > 0 && !mbar_wait(bar(L_OD), (it - 1) & 1, abort_flag)) return false;
                tc_fence_after();
#pragma unroll
                for (int ks = 0; ks < 4; ++ks) {
                    const uint64_t a = umma_smem_desc(base + L.off_p + b * kPBuf + ks * 32, 16, 1024);
                    const uint64_t v = umma_smem_desc(base + L.off_v + s * L.nv * kKBlk + ks * 2048, kKBlk, 1024);
                    umma_f16(tmem_o, a, v, id_pv, (!first || ks > 0) ? 1u : 0u);
                }
                umma_commit(bar(L_PV + b));
                umma_commit(bar(L_VE + s));
                if (last) umma_commit(bar(L_OF));
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
                if (!mbar_wait(bar(L_Q), i & 1, abort_flag)) { ok = false; break; }
                for (int j = 0; j < n_kt; ++j, ++gs) {
                    const int b = gs & 1, s = gs % NST;
                    if (!mbar_wait(bar(L_KF + s), (gs / NST) & 1, abort_flag)) { ok = false; break; }
                    if (gs >= 2 && !mbar_wait(bar(L_SE + b), ((gs >> 1) - 1) & 1, abort_flag)) { ok = false; break; }
                    tc_fence_after();
                    for (int blk = 0; blk < nq; ++blk)
#pragma unroll
                        for (int ks = 0; ks < 4; ++ks) {
                            const uint64_t a = umma_smem_desc(base + blk * kQBlk + ks * 32, 16, 1024);
                            const uint64_t k = umma_smem_desc(base + L.off_k + (s * nq + blk) * kKBlk + ks * 32, 16, 1024);
                            umma_f16(tmem + b * kLN, a, k, id_s, (blk > 0 || ks > 0) ? 1u : 0u);
                        }
                    umma_commit(bar(L_SF + b));
                    umma_commit(bar(L_KE + s));
                    if (j == n_kt - 1) umma_commit(bar(L_QE));
                    if (pending && !issue_pv(pg, pfirst, plast, pitem)) { ok = false; break; }
                    pending = true; pg = gs; pfirst = (j == 0); plast = (j == n_kt - 1); pitem = i;
                }
            }
            if (ok && pending) issue_pv(pg, pfirst, plast, pitem);
        }
    } else {
        // ------------------------------ softmax / correction / epilogue ------------------------------
        const int r = threadIdx.x & 127;                 // query row == TMEM lane
        const int hf = threadIdx.x >> 7;                 // which 32 of a tile's 64 keys / which half of each 64 output columns
        const int wrow = (warp & 3) * 32;
        const uint32_t lane_base = (uint32_t)wrow << 16;
        const int pair_bar = 1 + (warp & 3);             // named barrier shared by the two warps that cover the same rows
        const int W = L.window > 0 ? L.window : 1 << 30;
        const float sc = L.sc;
        bool ok = true;
        int gs = 0;
        for (int it = 0; it < n_my; ++it) {
            const Item im = item(it);
            const LatentTile& tile = im.t;
            const int q_pos = tile.q_pos0 + r, w_lo = tile.q_pos0 + wrow;     // this row's position, the warp's first
            float m_ref = -INFINITY, l = 0.f;
            for (int j = 0; j < im.n_kt; ++j, ++gs) {
                const int b = gs & 1;
                if (!mbar_wait_warp(bar(L_SF + b), (gs >> 1) & 1, abort_flag)) ok = false;
                tc_fence_after();
                uint32_t sr[32];
                tmem_ld32(tmem + lane_base + b * kLN + hf * 32, sr);
                tmem_wait_ld();
                tc_fence_before();
                mbar_arrive(bar(L_SE + b));
                const int col0 = im.key0 + j * kLN + hf * 32;
                float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
                if (col0 + 31 > w_lo || col0 <= w_lo + 31 - W) {              // warp-uniform: an edge may cross this half tile
                    const int hi = q_pos - col0, lo = hi - W;                 // visible: lo < c <= hi
#pragma unroll
                    for (int c = 0; c < 32; ++c) {
                        const float v = (c <= hi && c > lo) ? __uint_as_float(sr[c]) : -INFINITY;
                        sr[c] = __float_as_uint(v);
                        mx4[c & 3] = fmaxf(mx4[c & 3], v);
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < 32; ++c) mx4[c & 3] = fmaxf(mx4[c & 3], __uint_as_float(sr[c]));
                }
                float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
                x_mx[(b * 2 + hf) * 128 + r] = mx;
                asm volatile("bar.sync %0, 64;" ::"r"(pair_bar) : "memory");
                mx = fmaxf(mx, x_mx[(b * 2 + (hf ^ 1)) * 128 + r]) * sc;
                const float m_new = fmaxf(m_ref, mx);            // -inf while the row has seen no key
                const bool need = (m_new - m_ref > 8.0f);        // true at the row's first key (m_ref = -inf)
                if (__any_sync(0xffffffffu, need)) {             // same decision in both warps of the pair: same rows, same values
                    if (j > 0) {
                        if (!mbar_wait_warp(bar(L_PV + ((gs - 1) & 1)), ((gs - 1) >> 1) & 1, abort_flag)) ok = false;
                        tc_fence_after();
                        const float alpha = m_new == m_ref ? 1.0f : exp2f(m_ref - m_new);
                        l *= alpha;
#pragma unroll 1
                        for (int cc = 0; cc < L.nv; ++cc) {
                            uint32_t o[32];
                            tmem_ld32(tmem_o + lane_base + (2 * cc + hf) * 32, o);
                            tmem_wait_ld();
#pragma unroll
                            for (int c = 0; c < 32; ++c) o[c] = __float_as_uint(__uint_as_float(o[c]) * alpha);
                            tmem_st32(tmem_o + lane_base + (2 * cc + hf) * 32, o);
                        }
                        tmem_wait_st();
                    }
                    m_ref = m_new;
                }
                // P = 2^(s * scale - m_ref) as bf16 into the swizzled K-major A tile
                if (gs >= 2 && !mbar_wait_warp(bar(L_PV + b), ((gs >> 1) - 1) & 1, abort_flag)) ok = false;
                const float m_use = m_ref == -INFINITY ? 0.f : m_ref;
                unsigned char* prow = sm + L.off_p + b * kPBuf + r * 128;
                float ls4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int c8 = 0; c8 < 4; ++c8) {
                    uint32_t pk[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float p0 = ex2p(fmaf(__uint_as_float(sr[c8 * 8 + 2 * e]), sc, -m_use));
                        const float p1 = ex2p(fmaf(__uint_as_float(sr[c8 * 8 + 2 * e + 1]), sc, -m_use));
                        ls4[e] += p0 + p1;
                        pk[e] = pack_bf16x2(p0, p1);
                    }
                    *reinterpret_cast<uint4*>(prow + (((hf * 4 + c8) ^ (r & 7)) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                }
                l += (ls4[0] + ls4[1]) + (ls4[2] + ls4[3]);
                fence_proxy_async_smem();
                tc_fence_before();
                mbar_arrive(bar(L_PF + b));
            }
            // row sums of the two halves: through the exchange slot the next step will use, hence the second barrier
            float* x_l = x_mx + (gs & 1) * 256;
            x_l[hf * 128 + r] = l;
            asm volatile("bar.sync %0, 64;" ::"r"(pair_bar) : "memory");
            l += x_l[(hf ^ 1) * 128 + r];
            asm volatile("bar.sync %0, 64;" ::"r"(pair_bar) : "memory");
            // ---- output: full tiles through shared memory (the idle P buffers) and tiled TMA stores, others from registers ----
            const bool via_tma = tile.n_rows == kLM;
            if (!mbar_wait_warp(bar(L_OF), it & 1, abort_flag)) ok = false;
            tc_fence_after();
            const float inv_l = 1.0f / l;
#pragma unroll 1
            for (int k = 0; k < L.nv; ++k) {
                uint32_t o[32], h2[16];
                tmem_ld32(tmem_o + lane_base + (2 * k + hf) * 32, o);
                tmem_wait_ld();
                if (k == L.nv - 1) {           // this thread has read its part of O: the next item's first PV may overwrite it
                    tc_fence_before();
                    mbar_arrive(bar(L_OD));
                }
#pragma unroll
                for (int c = 0; c < 16; ++c) h2[c] = pack_bf16x2(__uint_as_float(o[2 * c]) * inv_l, __uint_as_float(o[2 * c + 1]) * inv_l);
                if (!via_tma) {
                    if (r < tile.n_rows && ok) {
                        __nv_bfloat16* dst = out + (size_t)(tile.q_row0 + r) * L.heads * L.nv * 64 + (im.head * L.nv + k) * 64 + hf * 32;
#pragma unroll
                        for (int q8 = 0; q8 < 4; ++q8)
                            *reinterpret_cast<uint4*>(dst + 8 * q8) = make_uint4(h2[4 * q8], h2[4 * q8 + 1], h2[4 * q8 + 2], h2[4 * q8 + 3]);
                    }
                    continue;
                }
                if (k >= 2) {                  // the store of round k - 2 must have read this buffer
                    if (threadIdx.x == 0) bulk_wait_group_read1();
                    asm volatile("bar.sync 5, 256;" ::: "memory");
                }
                unsigned char* srow = sm + L.off_p + (k & 1) * kPBuf + r * 128;
#pragma unroll
                for (int q8 = 0; q8 < 4; ++q8)
                    *reinterpret_cast<uint4*>(srow + (((hf * 4 + q8) ^ (r & 7)) << 4)) = make_uint4(h2[4 * q8], h2[4 * q8 + 1], h2[4 * q8 + 2], h2[4 * q8 + 3]);
                fence_proxy_async_smem();
                asm volatile("bar.sync 5, 256;" ::: "memory");
                if (threadIdx.x == 0 && ok) {
                    tma_store_2d(&map_o, base + L.off_p + (k & 1) * kPBuf, (im.head * L.nv + k) * 64, tile.q_row0);
                    bulk_commit_group();
                }
            }
            if (via_tma) {                     // the P buffers go back to the softmax of the next item
                if (threadIdx.x == 0) bulk_wait_group_read0();
                asm volatile("bar.sync 5, 256;" ::: "memory");
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
    if (threadIdx.x == 0 && *abort_flag) atomicExch(error_word, 4);
}

static uint32_t lp_smem(int nq, int nv, int stages) { return nq * kQBlk + stages * (nq + nv) * kKBlk + 2 * kPBuf + 256 + 2048; }

bool latent_prefill_fits(const LatentShape& sh) {
    const int nq = (sh.dp + sh.rp) / 64, nv = sh.vp / 64;
    return nq <= 4 && nv <= 4 && sh.rot > 0 && sh.scale > 0.f && lp_smem(nq, nv, 2) <= 227 * 1024;
}

// q [rows][heads][dp + rp], k [ctx][heads][dp], k_rot [ctx][rp], v [ctx][heads][vp], out [rows][heads][vp], all bf16.
int launch_latent_prefill(const LatentShape& sh, const void* q, int rows, const void* k, const void* k_rot, const void* v, int ctx_rows,
                          const LatentTile* d_tiles, int n_tiles, void* out, int* d_error, cudaStream_t s) {
    if (n_tiles <= 0) return 0;
    const int nd = sh.dp / 64, nr = sh.rp / 64, nv = sh.vp / 64, nq = nd + nr;
    auto map = [&](CUtensorMap* m, const void* p, int cols, int n, int box_rows) -> int {
        const uint64_t dims[2] = {(uint64_t)cols, (uint64_t)n};
        const uint64_t str[1] = {(uint64_t)cols * 2};
        const uint32_t box[2] = {64, (uint32_t)box_rows};
        return make_tensor_map(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p, dims, str, box);
    };
    CUtensorMap mq, mk, mr, mv, mo;
    B2_TRY(map(&mq, q, sh.q_cols(), rows, kLM));
    B2_TRY(map(&mk, k, sh.heads * sh.dp, ctx_rows, kLN));
    B2_TRY(map(&mr, k_rot, sh.rp, ctx_rows, kLN));
    B2_TRY(map(&mv, v, sh.heads * sh.vp, ctx_rows, kLN));
    B2_TRY(map(&mo, out, sh.heads * sh.vp, rows, kLM));
    static PerDeviceOnce once;
    B2_PER_DEVICE_ONCE(once,
        B2_CUDA(cudaFuncSetAttribute(latent_prefill_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        B2_CUDA(cudaFuncSetAttribute(latent_prefill_kernel<3>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024)));
    int n_sm = 0;
    B2_TRY(device_sm_count(&n_sm));
    const int stages = lp_smem(nq, nv, 3) <= 227 * 1024 ? 3 : 2, n_items = n_tiles * sh.heads;
    LpShape L{sh.heads, nd, nr, nv, sh.window, sh.scale * 1.4426950408889634f};
    L.off_k = nq * kQBlk;
    L.off_v = L.off_k + stages * nq * kKBlk;
    L.off_p = L.off_v + stages * nv * kKBlk;
    L.off_bar = L.off_p + 2 * kPBuf;
    auto go = [&](auto kernel) {
        kernel<<<std::min(n_items, n_sm), kLThreads, lp_smem(nq, nv, stages), s>>>(mq, mk, mr, mv, mo, L, d_tiles, n_items, (__nv_bfloat16*)out, d_error);
    };
    if (stages == 3) go(latent_prefill_kernel<3>); else go(latent_prefill_kernel<2>);
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
