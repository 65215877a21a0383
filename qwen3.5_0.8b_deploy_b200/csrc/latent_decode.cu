// Split decode attention over cached latents, up to 16 heads at a time (bf16).
//
// With absorbed queries all heads of a row share one key and value stream: the cache rows themselves.  A row of a decode
// step needs the pages its window touches; the pages of all (row, head group) pairs form one list that is cut into equal
// ranges, one per CTA (one CTA per SM), so every SM streams the same number of bytes whatever the lengths are.  A producer
// lane brings whole pages (64 rows) into a ring of shared-memory stages with bulk TMA copies; eight consumer warps run
//     S [16 heads x 64 keys] = Q' [16 x (rank + rot)] C^T     one 8-key tile per warp
//     O [16 x rank] += P C                                    rank / 8 columns per warp
// on mma.sync m16n8k16 (bf16, fp32 accumulation): at 16 query rows per key byte the kernel is bound by HBM, not by the
// tensor pipe.  A range that ends inside a pair leaves an (m, l, O) partial; the CTA that delivers a pair's last one joins
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
constexpr int kSPitch = 68;           // floats per row of the score tile

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

struct LdLayout { uint32_t q, s, mx, pre, bar, stage0, stage_bytes, total; int stages; };
__host__ __device__ inline LdLayout ld_layout(int pitch, int rows) {
    LdLayout L;
    L.q = 0;
    L.s = L.q + kHG * pitch * 2;
    L.s = (L.s + 127) / 128 * 128;
    L.mx = L.s + 2 * kHG * kSPitch * 4;
    L.pre = L.mx + 2 * 8 * kHG * 4;
    L.bar = L.pre + (rows + 2 + 3) / 4 * 16;
    L.bar = (L.bar + 15) / 16 * 16;
    L.stage0 = (L.bar + 96 + 127) / 128 * 128;
    L.stage_bytes = kPageTokens * pitch * 2;
    const uint32_t room = 227 * 1024 - 256 - L.stage0;       // the last column tile of a warp may read a little past a row's end
    L.stages = (int)(room / L.stage_bytes);
    if (L.stages > 4) L.stages = 4;
    L.total = L.stage0 + L.stages * L.stage_bytes + 256;
    return L;
}
struct Seg { int row, hg, p0, p1, np; };   // pages [p0, p1) of the np of one pair
}  // namespace

// NT = 8-column tiles of the latent per consumer warp
template <int NT>
__global__ void __launch_bounds__(kLdThreads, 1)
latent_decode_kernel(const LatentShape sh, const __nv_bfloat16* __restrict__ qa, const LatentView cache, const int* __restrict__ row_slot,
                     const int* __restrict__ row_pos, int rows, float* __restrict__ part, int* __restrict__ counters,
                     __nv_bfloat16* __restrict__ out, unsigned long long* stamp) {
    extern __shared__ __align__(128) unsigned char sm[];
    const int pitch = sh.row_pitch(), hgs = (sh.heads + kHG - 1) / kHG;
    const LdLayout L = ld_layout(pitch, rows);
    const uint32_t base = smem_u32(sm);
    int* s_pre = reinterpret_cast<int*>(sm + L.pre);              // pages before row r; [rows] = all; [rows + 1] = most of one row
    uint64_t* bars = reinterpret_cast<uint64_t*>(sm + L.bar);     // full[4], empty[4]
    volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + 8);
    int* s_last = reinterpret_cast<int*>(bars + 9);
    auto full = [&](int s) { return base + L.bar + 8u * s; };
    auto empty = [&](int s) { return base + L.bar + 32u + 8u * s; };
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int s = 0; s < 4; ++s) { mbar_init(full(s), 1); mbar_init(empty(s), 8); }
        *abort_flag = 0;
        mbar_fence_init();
    }
    pdl_wait();
    auto first_key = [&](int pos) { return sh.window > 0 ? max(0, pos - sh.window + 1) : 0; };
    if (warp == 0) {                                              // page counts and their running sum
        int sum = 0, most = 0;
        for (int r0 = 0; r0 < rows; r0 += 32) {
            const int r = r0 + lane;
            int n = 0;
            if (r < rows) {
                const int slot = row_slot[r], pos = row_pos[r];
                if (slot >= 0 && slot < cache.max_seqs && pos < cache.capacity[slot]) n = pos / kPageTokens - first_key(pos) / kPageTokens + 1;
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
            int it = 0;
            for (int u = u0; u < u1;) {
                const Seg g = segment(u);
                const int slot = row_slot[g.row], first = first_key(row_pos[g.row]) / kPageTokens;
                const int* table = cache.block_table + (size_t)slot * cache.max_pages_per_seq + first;
                for (int p = g.p0; p < g.p1; ++p, ++it) {
                    const int s = it % L.stages;
                    if (it >= L.stages && !mbar_wait(empty(s), (it / L.stages - 1) & 1, abort_flag)) { u = u1; break; }
                    mbar_arrive_expect_tx(full(s), L.stage_bytes);
                    bulk_g2s(base + L.stage0 + s * L.stage_bytes,
                             static_cast<const __nv_bfloat16*>(cache.rows) + (size_t)table[p] * kPageTokens * pitch, L.stage_bytes, full(s));
                }
                u += g.p1 - g.p0;
            }
        }
    } else {
        const int g4 = lane >> 2, t4 = lane & 3;                  // fragment row and column pair
        const int ksteps = (pitch - 8) / 16;
        const float sc = sh.scale * 1.4426950408889634f;
        const uint32_t a_addr = base + L.q + ((lane & 15) * pitch + (lane >> 4) * 8) * 2;
        int it = 0;
        for (int u = u0; u < u1;) {
            const Seg g = segment(u);
            u += g.p1 - g.p0;
            const int pos = row_pos[g.row], first = first_key(pos), key0 = first / kPageTokens * kPageTokens;
            const int n_heads = min(kHG, sh.heads - g.hg * kHG);
            sync_consumers();                                     // everyone has left the previous pair's queries
            {
                const uint4* src = reinterpret_cast<const uint4*>(qa + ((size_t)g.row * sh.heads + g.hg * kHG) * pitch);
                const int per_row = pitch / 8;
                for (int e = tid; e < kHG * per_row; e += 256)
                    reinterpret_cast<uint4*>(sm + L.q)[e] = e / per_row < n_heads ? src[e] : make_uint4(0u, 0u, 0u, 0u);
            }
            sync_consumers();
            float o[NT][4], m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
#pragma unroll
            for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
            for (int p = g.p0; p < g.p1; ++p, ++it) {
                const int s = it % L.stages, b = it & 1;
                const uint32_t st = base + L.stage0 + s * L.stage_bytes;
                mbar_wait_warp(full(s), (it / L.stages) & 1, abort_flag);
                // ---- scores of keys 8 warp .. 8 warp + 7 of the page ----
                float d[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
                const uint32_t b_addr = st + ((8 * warp + (lane & 7)) * pitch + (lane >> 3) * 8) * 2;
                int ks = 0;
#pragma unroll 4
                for (; ks + 1 < ksteps; ks += 2) {
                    uint32_t a0[4], a1[4], bb[4];
                    ldm_x4(bb, b_addr + ks * 32);
                    ldm_x4(a0, a_addr + ks * 32);
                    ldm_x4(a1, a_addr + ks * 32 + 32);
                    mma_bf16(d[0], a0, bb[0], bb[1]);
                    mma_bf16(d[1], a1, bb[2], bb[3]);
                }
                if (ks < ksteps) {                                // the last step reads 8 columns of the row's tail beside its own 16
                    uint32_t a0[4], bb[4];
                    ldm_x4(bb, st + ((8 * warp + (lane & 7)) * pitch + ((lane >> 3) & 1) * 8) * 2 + ks * 32);
                    ldm_x4(a0, a_addr + ks * 32);
                    mma_bf16(d[0], a0, bb[0], bb[1]);
                }
                float v[4];
                const int kpos = key0 + p * kPageTokens + 8 * warp + 2 * t4;
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int k = kpos + (e & 1);
                    v[e] = (k >= first && k <= pos) ? (d[0][e] + d[1][e]) * sc : -INFINITY;
                }
                float* S = reinterpret_cast<float*>(sm + L.s) + b * kHG * kSPitch;
                float* X = reinterpret_cast<float*>(sm + L.mx) + b * 8 * kHG;
                *reinterpret_cast<float2*>(S + g4 * kSPitch + 8 * warp + 2 * t4) = make_float2(v[0], v[1]);
                *reinterpret_cast<float2*>(S + (g4 + 8) * kSPitch + 8 * warp + 2 * t4) = make_float2(v[2], v[3]);
                float x0 = fmaxf(v[0], v[1]), x1 = fmaxf(v[2], v[3]);
#pragma unroll
                for (int k = 1; k < 4; k <<= 1) {
                    x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, k));
                    x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, k));
                }
                if (t4 == 0) { X[warp * kHG + g4] = x0; X[warp * kHG + g4 + 8] = x1; }
                sync_consumers();
                // ---- weights: every warp forms the whole 16 x 64 tile as its A operand ----
                float n0 = m0, n1 = m1;
#pragma unroll
                for (int w = 0; w < 8; ++w) { n0 = fmaxf(n0, X[w * kHG + g4]); n1 = fmaxf(n1, X[w * kHG + g4 + 8]); }
                const float al0 = ex2l(m0 - n0), al1 = ex2l(m1 - n1);   // a page holds a visible key, so n0 and n1 are finite
                m0 = n0; m1 = n1;
                l0 *= al0; l1 *= al1;
#pragma unroll
                for (int n = 0; n < NT; ++n) { o[n][0] *= al0; o[n][1] *= al0; o[n][2] *= al1; o[n][3] *= al1; }
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    uint32_t a[4];
#pragma unroll
                    for (int hh = 0; hh < 2; ++hh) {
                        const float2 s0 = *reinterpret_cast<const float2*>(S + g4 * kSPitch + 16 * k + 8 * hh + 2 * t4);
                        const float2 s1 = *reinterpret_cast<const float2*>(S + (g4 + 8) * kSPitch + 16 * k + 8 * hh + 2 * t4);
                        const float p0 = ex2l(s0.x - n0), p1 = ex2l(s0.y - n0), p2 = ex2l(s1.x - n1), p3 = ex2l(s1.y - n1);
                        l0 += p0 + p1; l1 += p2 + p3;
                        a[2 * hh] = pack_bf16x2(p0, p1);
                        a[2 * hh + 1] = pack_bf16x2(p2, p3);
                    }
                    // value tiles: 16 keys x 16 columns per transposed load
                    const uint32_t v_addr = st + ((16 * k + (lane & 15)) * pitch + warp * 8 * NT + (lane >> 4) * 8) * 2;
#pragma unroll
                    for (int n = 0; n < NT; n += 2) {
                        if (warp * 8 * NT + 8 * n >= sh.rank) break;      // tiles behind the latent: never stored, and past the stage's end
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
            for (int k = 1; k < 4; k <<= 1) {
                l0 += __shfl_xor_sync(0xffffffffu, l0, k);
                l1 += __shfl_xor_sync(0xffffffffu, l1, k);
            }
            const int col = warp * 8 * NT + 2 * t4;
            __nv_bfloat16* orow = out + ((size_t)g.row * sh.heads + g.hg * kHG) * sh.rank;
            if (g.p0 == 0 && g.p1 == g.np) {
                const float i0 = 1.f / l0, i1 = 1.f / l1;
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int hd = g4 + 8 * (e >> 1), c = col + 8 * n + (e & 1);
                        if (hd < n_heads && c < sh.rank) orow[(size_t)hd * sh.rank + c] = __float2bfloat16_rn(o[n][e] * (e < 2 ? i0 : i1));
                    }
                continue;
            }
            // ---- partial of a split pair: slot = this CTA's place among the CTAs that share it ----
            const int pair = g.row * hgs + g.hg, begin = s_pre[g.row] * hgs + g.hg * g.np, end = begin + g.np;
            const int cta0 = begin / per, n_parts = (end - 1) / per - cta0 + 1, ld = sh.rank + 2;
            float* dst = part + ((size_t)pair * kLdParts + (blockIdx.x - cta0)) * kHG * ld;
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int hd = g4 + 8 * (e >> 1), c = col + 8 * n + (e & 1);
                    if (c < sh.rank) dst[hd * ld + c] = o[n][e];
                }
            if (warp == 0 && t4 == 0) {
                dst[g4 * ld + sh.rank] = m0; dst[g4 * ld + sh.rank + 1] = l0;
                dst[(g4 + 8) * ld + sh.rank] = m1; dst[(g4 + 8) * ld + sh.rank + 1] = l1;
            }
            __threadfence();
            sync_consumers();
            if (tid == 0) {
                const int seen = atomicAdd(counters + pair, 1);
                *s_last = seen == n_parts - 1;
                if (seen == n_parts - 1) counters[pair] = 0;      // ready for the next launch
            }
            sync_consumers();
            if (*s_last) {
                __threadfence();
                const float* src = part + (size_t)pair * kLdParts * kHG * ld;
                for (int e = tid; e < n_heads * sh.rank; e += 256) {
                    const int hd = e / sh.rank, c = e % sh.rank;
                    float mx = -INFINITY, l = 0.f, acc = 0.f;
                    for (int q = 0; q < n_parts; ++q) mx = fmaxf(mx, __ldcg(src + ((size_t)q * kHG + hd) * ld + sh.rank));
                    for (int q = 0; q < n_parts; ++q) {
                        const float* r = src + ((size_t)q * kHG + hd) * ld;
                        const float w = ex2l(__ldcg(r + sh.rank) - mx);
                        l += w * __ldcg(r + sh.rank + 1);
                        acc += w * __ldcg(r + c);
                    }
                    orow[(size_t)hd * sh.rank + c] = __float2bfloat16_rn(acc / l);
                }
            }
        }
    }
    __syncthreads();
    stamp_end(stamp);
    if (tid == 0 && *abort_flag) atomicExch(cache.error, 3);
}

bool latent_decode_fits(const LatentShape& sh, int max_rows) {
    return sh.rank <= 512 && max_rows <= kLdMaxRows && ld_layout(sh.row_pitch(), max_rows).stages >= 2;
}

size_t latent_decode_scratch_floats(const LatentShape& sh, int max_rows) {
    return (size_t)max_rows * ceil_div(sh.heads, kHG) * kLdParts * kHG * (sh.rank + 2);
}

int launch_latent_decode(const LatentShape& sh, const void* qa, const LatentView& cache, const int* row_slot, const int* row_pos, int rows,
                         float* part, int* counters, void* out, cudaStream_t s) {
    int n_sm = 0;
    B2_TRY(device_sm_count(&n_sm));
    const uint32_t smem = ld_layout(sh.row_pitch(), rows).total;
    static PerDeviceOnce once;
    B2_PER_DEVICE_ONCE(once,
        B2_CUDA(cudaFuncSetAttribute(latent_decode_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        B2_CUDA(cudaFuncSetAttribute(latent_decode_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        B2_CUDA(cudaFuncSetAttribute(latent_decode_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        B2_CUDA(cudaFuncSetAttribute(latent_decode_kernel<8>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024)));
    unsigned long long* stamp = prof_stamp_slot(PROF_FA_DECODE);
    auto go = [&](auto kernel) {
        launch_pdl(kernel, dim3(n_sm), dim3(kLdThreads), smem, s, sh, (const __nv_bfloat16*)qa, cache, row_slot, row_pos, rows, part, counters,
                   (__nv_bfloat16*)out, stamp);
    };
    if (sh.rank <= 64) go(latent_decode_kernel<1>);
    else if (sh.rank <= 128) go(latent_decode_kernel<2>);
    else if (sh.rank <= 256) go(latent_decode_kernel<4>);
    else go(latent_decode_kernel<8>);
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
