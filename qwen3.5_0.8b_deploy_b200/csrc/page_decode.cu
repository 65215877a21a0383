// Split decode attention over pages of cache rows, 16 query rows at a time (bf16).
//
// Latents: with absorbed queries all heads of a row share one key and value stream, the cache rows themselves, whose first
// `rank` columns are the values; 16 heads form a group.  Differential attention: a group is one key / value head with up to 8
// query heads; its cache rows are [k of map 1 | k of map 2 | v], and its query rows 0 .. 7 hold the heads' map-1 queries over
// the columns of map 1 (zeros elsewhere), rows 8 .. 15 the map-2 queries over those of map 2, so that one product gives the
// scores of both maps and one product both maps' outputs, which meet in the same thread.
//
// A row of a decode step needs the pages its kept positions and its window touch; the pages of all (row, group) pairs form one
// list that is cut into equal ranges, one per CTA (one CTA per SM), so every SM streams the same number of bytes whatever the
// lengths are.  A producer lane brings whole pages (64 rows) into a ring of shared-memory stages with bulk TMA copies; eight
// consumer warps run
//     S [16 x 64 keys] = Q [16 x key columns] K^T     a quarter of the contraction for half of the keys per warp
//     O [16 x value columns] += P V                   an eighth of the columns per warp
// on mma.sync m16n8k16 (bf16, fp32 accumulation): at 16 query rows per key byte the kernel is bound by HBM, not by the
// tensor pipe.  What counts on chip is shared-memory traffic: a warp keeps its part of the queries in registers for a whole
// pair and every key and value byte is read once; the four partial scores meet in the softmax step, which 16 threads per
// head do once for all warps.  A range that ends inside a pair leaves an (m, l, O) partial; the CTA that delivers a pair's last one joins
// them.  The row pitch is an odd number of 16-byte units, which keeps ldmatrix free of bank conflicts.
#include "block_model.cuh"
#include "elem.cuh"
#include "ptx_utils.cuh"

#include <algorithm>

namespace b200 {

namespace {
constexpr int kHG = 16;               // heads per group
constexpr int kLdParts = 16;          // partial slots per pair
constexpr int kLdMaxRows = 2048;
constexpr int kLdThreads = 288;       // 8 consumer warps + producer
constexpr int kSPitch = 68;           // floats per row of a score tile
constexpr int kPPitch = 72;           // bf16 per row of the weight tile

__device__ __forceinline__ void ldm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldm_x4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2l(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void sync_consumers() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// What the kernel is told about the rows it reads.
struct LdShape {
    int pitch, qpitch;                    // elements per cache row of a group / per query row
    int groups;                           // groups per row
    int ksteps, vcol0, vcols;             // 16-column steps of the contraction; value columns
    int window, keep;
    float sc;                             // score factor times log2 e
    int heads, per;                       // heads of a row, of a group
    int vdim;                             // differential attention: real value columns, and the constants of the combination
    float lambda, out_scale, eps;
};
struct LdLayout { uint32_t q, q_bytes, s, p, pre, bar, stage0, stage_bytes, total; int stages; };
__host__ __device__ inline LdLayout ld_layout(int pitch, int qpitch, int rows) {
    LdLayout L;
    L.q = 0;
    L.q_bytes = (kHG * qpitch * 2 + 127) / 128 * 128;        // two query buffers
    L.s = L.q + 2 * L.q_bytes;
    L.p = L.s + 4 * kHG * kSPitch * 4;                       // partial scores of the four quarters
    L.pre = L.p + kHG * kPPitch * 2 + 3 * kHG * 4 + 64 * 4;  // weights (bf16), then factor, maximum and sum of every query row, sums of squares
    L.bar = L.pre + (2 * rows + 2 + 3) / 4 * 16;
    L.bar = (L.bar + 15) / 16 * 16;
    L.stage0 = (L.bar + 128 + 127) / 128 * 128;
    L.stage_bytes = kPageTokens * pitch * 2;
    const uint32_t room = 227 * 1024 - 256 - L.stage0;       // the last column tile of a warp may read a little past a row's end
    L.stages = (int)(room / L.stage_bytes);
    if (L.stages > 4) L.stages = 4;
    L.total = L.stage0 + L.stages * L.stage_bytes + 256;
    return L;
}
template <int NT> constexpr int kPartFloats = NT * 1024 + 32;      // O in register order, then (m, l) of the 16 heads
struct Seg { int row, hg, p0, p1, np; };   // pages [p0, p1) of the np of one pair
// The pages of a row: those with kept positions, then those its window touches behind them.
struct Pages {
    int first, kept, w0, n;               // first position of the window, pages of kept positions, first page behind them, pages in all
    __device__ Pages(const LdShape& sh, int pos) {
        first = sh.window > 0 ? max(0, pos - sh.window + 1) : 0;
        kept = (min(sh.keep, pos + 1) + kPageTokens - 1) / kPageTokens;
        w0 = max(kept, first / kPageTokens);
        n = kept + max(0, pos / kPageTokens - w0 + 1);
    }
    __device__ int at(int j) const { return j < kept ? j : w0 + j - kept; }
};
}  // namespace

// NT = 8-column tiles of the latent per consumer warp, KQ = 16-column steps of the contraction per warp
template <int NT, int KQ, bool kDiff>
__global__ void __launch_bounds__(kLdThreads, 1)
page_decode_kernel(const LdShape sh, const __nv_bfloat16* __restrict__ qa, const LatentView cache, const int* __restrict__ row_slot,
                     const int* __restrict__ row_pos, int rows, float* __restrict__ part, int* __restrict__ counters,
                     __nv_bfloat16* __restrict__ out, unsigned long long* stamp) {
    extern __shared__ __align__(128) unsigned char sm[];
    const int pitch = sh.pitch, qpitch = sh.qpitch, hgs = sh.groups;
    const LdLayout L = ld_layout(pitch, qpitch, rows);
    const uint32_t base = smem_u32(sm);
    int* s_pre = reinterpret_cast<int*>(sm + L.pre);              // pages before row r; [rows] = all; [rows + 1] = most of one row
    int* s_pos = s_pre + rows + 2;
    uint64_t* bars = reinterpret_cast<uint64_t*>(sm + L.bar);     // full[4], empty[4], q_full[2], q_empty[2]
    volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + 12);
    int* s_last = reinterpret_cast<int*>(bars + 13);
    auto full = [&](int s) { return base + L.bar + 8u * s; };
    auto empty = [&](int s) { return base + L.bar + 32u + 8u * s; };
    auto q_full = [&](int b) { return base + L.bar + 64u + 8u * b; };
    auto q_empty = [&](int b) { return base + L.bar + 80u + 8u * b; };
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int s = 0; s < 4; ++s) { mbar_init(full(s), 1); mbar_init(empty(s), 8); }
        for (int b = 0; b < 2; ++b) { mbar_init(q_full(b), 1); mbar_init(q_empty(b), 8); }
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (!kDiff && sh.heads % kHG) {   // query rows of absent heads are never copied: finite from the start
        for (uint32_t e = tid; e < 2 * L.q_bytes / 16; e += kLdThreads) reinterpret_cast<uint4*>(sm + L.q)[e] = make_uint4(0u, 0u, 0u, 0u);
        fence_proxy_async_smem();
    }
    pdl_wait();
    if (warp == 0) {                                              // page counts and their running sum
        int sum = 0, most = 0;
        for (int r0 = 0; r0 < rows; r0 += 32) {
            const int r = r0 + lane;
            int n = 0;
            if (r < rows) {
                const int slot = row_slot[r], pos = row_pos[r];
                s_pos[r] = pos;
                if (slot >= 0 && slot < cache.max_seqs && pos < cache.capacity[slot]) n = Pages(sh, pos).n;
            }
            most = max(most, n);
            int inc = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int x = __shfl_up_sync(0xffffffffu, inc, o);
                if (lane >= o) inc += x;
            }
            if (r < rows) s_pre[r] = sum + inc - n;
            sum += __shfl_sync(0xffffffffu, inc, 31);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) most = max(most, __shfl_xor_sync(0xffffffffu, most, o));
        if (lane == 0) { s_pre[rows] = sum; s_pre[rows + 1] = most; }
    }
    __syncthreads();
    pdl_launch_dependents();
    stamp_begin(stamp);
    const int total = s_pre[rows] * hgs;
    const int per = max((total + (int)gridDim.x - 1) / (int)gridDim.x, (s_pre[rows + 1] + kLdParts - 2) / (kLdParts - 1));
    const int u0 = min(total, (int)blockIdx.x * per), u1 = min(total, u0 + per);
    auto segment = [&](int u) -> Seg {                            // the pair that unit u falls into, cut at u1
        int lo = 0, hi = rows - 1;
        while (lo < hi) {
            const int mid = (lo + hi + 1) >> 1;
            if (s_pre[mid] * hgs <= u) lo = mid; else hi = mid - 1;
        }
        Seg g;
        g.row = lo;
        g.np = s_pre[lo + 1] - s_pre[lo];
        const int off = u - s_pre[lo] * hgs;
        g.hg = off / g.np;
        g.p0 = off % g.np;
        g.p1 = min(g.np, g.p0 + (u1 - u));
        return g;
    };

    if (warp == 8) {
        if (lane == 0) {
            int it = 0, sg = 0;
            for (int u = u0; u < u1; ++sg) {
                const Seg g = segment(u);
                const int slot = row_slot[g.row];
                const Pages pg(sh, s_pos[g.row]);
                const uint32_t qb = (uint32_t)(kDiff ? kHG : min(kHG, sh.heads - g.hg * kHG)) * qpitch * 2;
                if (sg >= 2 && !mbar_wait(q_empty(sg & 1), ((sg >> 1) - 1) & 1, abort_flag)) break;
                mbar_arrive_expect_tx(q_full(sg & 1), qb);
                bulk_g2s(base + L.q + (sg & 1) * L.q_bytes, qa + (kDiff ? ((size_t)g.row * hgs + g.hg) * kHG : (size_t)g.row * sh.heads + g.hg * kHG) * qpitch, qb, q_full(sg & 1));
                const int* table = cache.block_table + (size_t)slot * cache.max_pages_per_seq;
                for (int p = g.p0; p < g.p1; ++p, ++it) {
                    const int s = it % L.stages;
                    if (it >= L.stages && !mbar_wait(empty(s), (it / L.stages - 1) & 1, abort_flag)) { u = u1; break; }
                    mbar_arrive_expect_tx(full(s), L.stage_bytes);
                    bulk_g2s(base + L.stage0 + s * L.stage_bytes,
                             static_cast<const __nv_bfloat16*>(cache.rows) + (kDiff ? (size_t)table[pg.at(p)] * hgs + g.hg : (size_t)table[pg.at(p)]) * kPageTokens * pitch,
                             L.stage_bytes, full(s));
                }
                u += g.p1 - g.p0;
            }
        }
    } else {
        const int g4 = lane >> 2, t4 = lane & 3;                  // fragment row and column pair
        const int ksteps = sh.ksteps, k0 = (warp & 3) * KQ, keys = (warp >> 2) * 32;
        const int srow = tid >> 4, skey = 4 * (tid & 15);         // softmax: head and four keys of this thread
        const float sc = sh.sc;
        float* SP = reinterpret_cast<float*>(sm + L.s);
        __nv_bfloat16* PT = reinterpret_cast<__nv_bfloat16*>(sm + L.p);
        float* s_al = reinterpret_cast<float*>(sm + L.p + kHG * kPPitch * 2);
        float *s_m = s_al + kHG, *s_l = s_m + kHG, *s_ss = s_l + kHG;      // s_ss: [8 warps][8 heads]
        const uint32_t p_addr = base + L.p + ((lane & 15) * kPPitch + (lane >> 4) * 8) * 2;
        int it = 0, sg = 0;
        for (int u = u0; u < u1; ++sg) {
            const Seg g = segment(u);
            u += g.p1 - g.p0;
            const int pos = s_pos[g.row];
            const Pages pg(sh, pos);
            const int n_heads = kDiff ? sh.per : min(kHG, sh.heads - g.hg * kHG);
            mbar_wait_warp(q_full(sg & 1), (sg >> 1) & 1, abort_flag);
            uint32_t qf[KQ][4];
            {
                const uint32_t a_addr = base + L.q + (sg & 1) * L.q_bytes + ((lane & 15) * qpitch + (lane >> 4) * 8) * 2;
#pragma unroll
                for (int k = 0; k < KQ; ++k)
                    if (k0 + k < ksteps) ldm_x4(qf[k], a_addr + (k0 + k) * 32);
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(q_empty(sg & 1));
            float o[NT][4], m_run = -INFINITY, l_run = 0.f;
#pragma unroll
            for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
            for (int p = g.p0; p < g.p1; ++p, ++it) {
                const int s = it % L.stages;
                const uint32_t st = base + L.stage0 + s * L.stage_bytes;
                mbar_wait_warp(full(s), (it / L.stages) & 1, abort_flag);
                // ---- partial scores of 32 keys over this warp's columns ----
                {
                    float d[4][4];
#pragma unroll
                    for (int n = 0; n < 4; ++n) d[n][0] = d[n][1] = d[n][2] = d[n][3] = 0.f;
                    const uint32_t b_addr = st + ((keys + (lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 8 + k0 * 16) * 2;
#pragma unroll
                    for (int k = 0; k < KQ; ++k)
                        if (k0 + k < ksteps) {
                            uint32_t b0[4], b1[4];
                            ldm_x4(b0, b_addr + k * 32);
                            ldm_x4(b1, b_addr + k * 32 + 32 * pitch);
                            mma_bf16(d[0], qf[k], b0[0], b0[1]);
                            mma_bf16(d[1], qf[k], b0[2], b0[3]);
                            mma_bf16(d[2], qf[k], b1[0], b1[1]);
                            mma_bf16(d[3], qf[k], b1[2], b1[3]);
                        }
                    float* S = SP + (warp & 3) * kHG * kSPitch + keys + 2 * t4;
#pragma unroll
                    for (int n = 0; n < 4; ++n) {
                        *reinterpret_cast<float2*>(S + g4 * kSPitch + 8 * n) = make_float2(d[n][0], d[n][1]);
                        *reinterpret_cast<float2*>(S + (g4 + 8) * kSPitch + 8 * n) = make_float2(d[n][2], d[n][3]);
                    }
                }
                sync_consumers();
                // ---- softmax: 16 threads per head ----
                {
                    const float* S = SP + srow * kSPitch + skey;
                    const float4 a = *reinterpret_cast<const float4*>(S), b = *reinterpret_cast<const float4*>(S + kHG * kSPitch);
                    const float4 c = *reinterpret_cast<const float4*>(S + 2 * kHG * kSPitch), d = *reinterpret_cast<const float4*>(S + 3 * kHG * kSPitch);
                    float v[4] = {(a.x + b.x) + (c.x + d.x), (a.y + b.y) + (c.y + d.y), (a.z + b.z) + (c.z + d.z), (a.w + b.w) + (c.w + d.w)};
                    const int kpos = pg.at(p) * kPageTokens + skey;
                    float mx = -INFINITY;
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        v[e] = ((kpos + e >= pg.first || kpos + e < sh.keep) && kpos + e <= pos) ? v[e] * sc : -INFINITY;
                        mx = fmaxf(mx, v[e]);
                    }
#pragma unroll
                    for (int k = 8; k > 0; k >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, k));
                    const float mn = fmaxf(m_run, mx), al = ex2l(m_run - mn);    // a page holds a visible key, so mn is finite
                    m_run = mn;
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[e] = ex2l(v[e] - mn);
                    l_run = l_run * al + ((v[0] + v[1]) + (v[2] + v[3]));
                    *reinterpret_cast<uint2*>(PT + srow * kPPitch + skey) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
                    if (skey == 0) s_al[srow] = al;
                }
                sync_consumers();
                // ---- O += P C over this warp's columns ----
                const float al0 = s_al[g4], al1 = s_al[g4 + 8];
#pragma unroll
                for (int n = 0; n < NT; ++n) { o[n][0] *= al0; o[n][1] *= al0; o[n][2] *= al1; o[n][3] *= al1; }
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    uint32_t a[4];
                    ldm_x4(a, p_addr + k * 32);
                    // value tiles: 16 keys x 16 columns per transposed load
                    const uint32_t v_addr = st + ((16 * k + (lane & 15)) * pitch + sh.vcol0 + warp * 8 * NT + (lane >> 4) * 8) * 2;
#pragma unroll
                    for (int n = 0; n < NT; n += 2) {
                        if (warp * 8 * NT + 8 * n >= sh.vcols) break;     // tiles behind the values: never stored, and past the stage's end
                        uint32_t bb[4];
                        ldm_x4_t(bb, v_addr + n * 16);
                        mma_bf16(o[n], a, bb[0], bb[1]);
                        if (n + 1 < NT) mma_bf16(o[n + 1], a, bb[2], bb[3]);
                    }
                }
                __syncwarp();
                if (lane == 0) mbar_arrive(empty(s));
            }
#pragma unroll
            for (int k = 8; k > 0; k >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, k);
            if (skey == 0) { s_m[srow] = m_run; s_l[srow] = l_run; }
            sync_consumers();
            float m0 = s_m[g4], m1 = s_m[g4 + 8], l0 = s_l[g4], l1 = s_l[g4 + 8];
            auto store = [&] {
                const float i0 = 1.f / l0, i1 = 1.f / l1;
                const int col = warp * 8 * NT + 2 * t4;
                if constexpr (kDiff) {            // rows g4 and g4 + 8 are the two maps of one head
                    float ss = 0.f;
#pragma unroll
                    for (int n = 0; n < NT; ++n) {
                        const bool in = warp * 8 * NT + 8 * n < sh.vcols;
                        o[n][0] = in ? o[n][0] * i0 - sh.lambda * (o[n][2] * i1) : 0.f;
                        o[n][1] = in ? o[n][1] * i0 - sh.lambda * (o[n][3] * i1) : 0.f;
                        ss += o[n][0] * o[n][0] + o[n][1] * o[n][1];
                    }
                    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
                    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
                    if (t4 == 0) s_ss[warp * 8 + g4] = ss;
                    sync_consumers();
                    ss = 0.f;
#pragma unroll
                    for (int w = 0; w < 8; ++w) ss += s_ss[w * 8 + g4];
                    const float f = sh.out_scale / sqrtf(ss / (float)sh.vdim + sh.eps);
                    if (g4 >= n_heads) return;
                    __nv_bfloat16* dst = out + ((size_t)g.row * sh.heads + g.hg * sh.per + g4) * sh.vcols + col;
#pragma unroll
                    for (int n = 0; n < NT; ++n)
                        if (col + 8 * n < sh.vcols) *reinterpret_cast<uint32_t*>(dst + 8 * n) = pack_bf16x2(o[n][0] * f, o[n][1] * f);
                    return;
                }
                __nv_bfloat16* orow = out + ((size_t)g.row * sh.heads + g.hg * kHG) * sh.vcols;
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int hd = g4 + 8 * e, c = col + 8 * n;
                        const float x = o[n][2 * e] * (e ? i1 : i0), y = o[n][2 * e + 1] * (e ? i1 : i0);
                        if (hd >= n_heads) continue;
                        __nv_bfloat16* dst = orow + (size_t)hd * sh.vcols + c;
                        if ((sh.vcols & 1) == 0) {
                            if (c < sh.vcols) *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(x, y);
                        } else {
                            if (c < sh.vcols) dst[0] = __float2bfloat16_rn(x);
                            if (c + 1 < sh.vcols) dst[1] = __float2bfloat16_rn(y);
                        }
                    }
            };
            if (g.p0 == 0 && g.p1 == g.np) { store(); continue; }
            // ---- partial of a split pair: slot = this CTA's place among the CTAs that share it; accumulators in register order ----
            const int pair = g.row * hgs + g.hg, begin = s_pre[g.row] * hgs + g.hg * g.np, end = begin + g.np;
            const int cta0 = begin / per, n_parts = (end - 1) / per - cta0 + 1, mine = blockIdx.x - cta0;
            float* pp = part + (size_t)pair * kLdParts * kPartFloats<NT>;
            {
                float* dst = pp + (size_t)mine * kPartFloats<NT>;
#pragma unroll
                for (int n = 0; n < NT; ++n) __stcg(reinterpret_cast<float4*>(dst) + n * 256 + tid, make_float4(o[n][0], o[n][1], o[n][2], o[n][3]));
                if (warp == 0 && t4 == 0) {
                    __stcg(reinterpret_cast<float2*>(dst + NT * 1024) + g4, make_float2(m0, l0));
                    __stcg(reinterpret_cast<float2*>(dst + NT * 1024) + g4 + 8, make_float2(m1, l1));
                }
            }
            __threadfence();
            sync_consumers();
            if (tid == 0) {
                const int seen = atomicAdd(counters + pair, 1);
                *s_last = seen == n_parts - 1;
                if (seen == n_parts - 1) counters[pair] = 0;      // ready for the next launch
                __threadfence();
            }
            sync_consumers();
            if (*s_last) {                                        // join the others' partials with the one still in registers
                auto join = [&](float2 a, float2 c, const float4 (&x)[NT]) {
                    const float n0 = fmaxf(m0, a.x), n1 = fmaxf(m1, c.x);
                    const float s0 = ex2l(m0 - n0), s1 = ex2l(m1 - n1), t0 = ex2l(a.x - n0), t1 = ex2l(c.x - n1);
                    m0 = n0; m1 = n1;
                    l0 = l0 * s0 + a.y * t0; l1 = l1 * s1 + c.y * t1;
#pragma unroll
                    for (int n = 0; n < NT; ++n) {
                        o[n][0] = o[n][0] * s0 + x[n].x * t0; o[n][1] = o[n][1] * s0 + x[n].y * t0;
                        o[n][2] = o[n][2] * s1 + x[n].z * t1; o[n][3] = o[n][3] * s1 + x[n].w * t1;
                    }
                };
                auto fetch = [&](int q, float2& a, float2& c, float4 (&x)[NT]) {
                    const float* src = pp + (size_t)q * kPartFloats<NT>;
                    a = __ldcg(reinterpret_cast<const float2*>(src + NT * 1024) + g4);
                    c = __ldcg(reinterpret_cast<const float2*>(src + NT * 1024) + g4 + 8);
#pragma unroll
                    for (int n = 0; n < NT; ++n) x[n] = __ldcg(reinterpret_cast<const float4*>(src) + n * 256 + tid);
                };
                for (int i = 0; i < n_parts - 1; i += 2) {        // two parts' loads under way together
                    const int qa2 = i + (i >= mine), qb2 = i + 1 + (i + 1 >= mine);
                    float2 a, c, b = make_float2(0.f, 0.f), d = b;
                    float4 x[NT], z[NT];
                    fetch(qa2, a, c, x);
                    if (i + 1 < n_parts - 1) fetch(qb2, b, d, z);
                    join(a, c, x);
                    if (i + 1 < n_parts - 1) join(b, d, z);
                }
                store();
            }
        }
    }
    __syncthreads();
    stamp_end(stamp);
    if (tid == 0 && *abort_flag) atomicExch(cache.error, 3);
}

static int ld_tiles(int vcols) { return vcols <= 64 ? 1 : vcols <= 128 ? 2 : vcols <= 256 ? 4 : 8; }

static bool page_decode_fits(const LdShape& sh, int max_rows) {
    return sh.vcols <= 512 && sh.ksteps <= 48 && max_rows <= kLdMaxRows && ld_layout(sh.pitch, sh.qpitch, max_rows).stages >= 2;
}

template <bool kDiff>
static int launch_page_decode(const LdShape& sh, const void* qa, const LatentView& cache, const int* row_slot, const int* row_pos, int rows, float* part,
                              int* counters, void* out, cudaStream_t s) {
    int n_sm = 0;
    B2_TRY(device_sm_count(&n_sm));
    const uint32_t smem = ld_layout(sh.pitch, sh.qpitch, rows).total;
    unsigned long long* stamp = prof_stamp_slot(PROF_FA_DECODE);
    auto go = [&](auto kernel) {
        launch_pdl(kernel, dim3(n_sm), dim3(kLdThreads), smem, s, sh, (const __nv_bfloat16*)qa, cache, row_slot, row_pos, rows, part, counters,
                   (__nv_bfloat16*)out, stamp);
    };
    auto pick = [&](auto nt) -> int {
        constexpr int NT = decltype(nt)::value;
        static PerDeviceOnce once;
        B2_PER_DEVICE_ONCE(once,
            B2_CUDA(cudaFuncSetAttribute(page_decode_kernel<NT, 3, kDiff>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
            B2_CUDA(cudaFuncSetAttribute(page_decode_kernel<NT, 9, kDiff>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
            B2_CUDA(cudaFuncSetAttribute(page_decode_kernel<NT, 12, kDiff>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024)));
        const int kq = ceil_div(sh.ksteps, 4);                    // contraction steps per warp
        if (kq <= 3) go(page_decode_kernel<NT, 3, kDiff>);
        else if (kq <= 9) go(page_decode_kernel<NT, 9, kDiff>);
        else go(page_decode_kernel<NT, 12, kDiff>);
        return 0;
    };
    switch (ld_tiles(sh.vcols)) {
        case 1: B2_TRY(pick(std::integral_constant<int, 1>{})); break;
        case 2: B2_TRY(pick(std::integral_constant<int, 2>{})); break;
        case 4: B2_TRY(pick(std::integral_constant<int, 4>{})); break;
        default: B2_TRY(pick(std::integral_constant<int, 8>{})); break;
    }
    B2_LAUNCH_CHECK();
    return 0;
}

constexpr float kLdLog2e = 1.4426950408889634f;

static LdShape latent_rows(const LatentShape& sh) {
    LdShape r{};
    r.pitch = r.qpitch = sh.row_pitch();
    r.groups = ceil_div(sh.heads, kHG);
    r.ksteps = (sh.row_pitch() - 8) / 16;
    r.vcols = sh.rank;
    r.window = sh.window;
    r.sc = sh.scale * kLdLog2e;
    r.heads = sh.heads;
    r.per = kHG;
    return r;
}

bool latent_decode_fits(const LatentShape& sh, int max_rows) { return page_decode_fits(latent_rows(sh), max_rows); }

size_t latent_decode_scratch_floats(const LatentShape& sh, int max_rows) {
    return (size_t)max_rows * ceil_div(sh.heads, kHG) * kLdParts * (ld_tiles(sh.rank) * 1024 + 32);
}

int launch_latent_decode(const LatentShape& sh, const void* qa, const LatentView& cache, const int* row_slot, const int* row_pos, int rows,
                         float* part, int* counters, void* out, cudaStream_t s) {
    return launch_page_decode<false>(latent_rows(sh), qa, cache, row_slot, row_pos, rows, part, counters, out, s);
}

static LdShape diff_rows(const DiffShape& sh, float lambda) {
    LdShape r{};
    r.pitch = sh.hp();
    r.qpitch = sh.qp();
    r.groups = sh.kv_heads;
    r.ksteps = 2 * sh.dp / 16;
    r.vcol0 = 2 * sh.dp;
    r.vcols = sh.vp;
    r.window = sh.window;
    r.keep = sh.keep;
    r.sc = sh.scale * kLdLog2e;
    r.heads = sh.heads;
    r.per = sh.heads / sh.kv_heads;
    r.vdim = sh.vdim;
    r.lambda = lambda;
    r.out_scale = 1.0f - sh.diff;
    r.eps = sh.eps;
    return r;
}

bool diff_decode_fits(const DiffShape& sh, int max_rows) { return sh.heads / sh.kv_heads <= 8 && page_decode_fits(diff_rows(sh, 0.f), max_rows); }

size_t diff_decode_scratch_floats(const DiffShape& sh, int max_rows) {
    return (size_t)max_rows * sh.kv_heads * kLdParts * (ld_tiles(sh.vp) * 1024 + 32);
}

int launch_diff_decode(const DiffShape& sh, float lambda, const void* qd, const LatentView& cache, const int* row_slot, const int* row_pos, int rows,
                       float* part, int* counters, void* out, cudaStream_t s) {
    return launch_page_decode<true>(diff_rows(sh, lambda), qd, cache, row_slot, row_pos, rows, part, counters, out, s);
}

}  // namespace b200
