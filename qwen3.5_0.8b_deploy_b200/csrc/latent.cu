// Attention over cached latents: the step behind the input projection (rotation, latent norm, append), the staging of a
// pass's context rows, and the absorbed attention of any size.
//
// A token's cache row is [latent c | rotated key part | zeros].  With the up-projections absorbed, q'_h = W_uk,h^T q_h (the
// unrotated part) and the rotated part of q, a score is q' . row, and the output of a head is W_uv,h (sum of weights x c).
#include "block_model.cuh"
#include "elem.cuh"
#include "ptx_utils.cuh"

#include <algorithm>

namespace b200 {

// The queries of a row: unrotated parts converted, rotated parts turned.  A warp per head.  With heads of up to 128 + 64
// columns (kSmallHead) two whole heads are requested before the first value is used; the others go piece by piece.
template <typename T, bool kSmallHead>
__device__ __forceinline__ void latent_queries(const LatentPreArgs& a, int row, const float* __restrict__ pr) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int half = a.sh.rot / 2, heads = a.sh.heads, dp = a.sh.dp, hw = a.sh.dp + a.sh.rp, ap = a.sh.row_pitch();
    const float2* __restrict__ cs = a.cs + (size_t)row * half;
    T* __restrict__ q = static_cast<T*>(a.q) + (size_t)row * heads * hw;
    T* __restrict__ qa = a.qa ? static_cast<T*>(a.qa) + (size_t)row * heads * ap + a.sh.rank : nullptr;
    auto rotated = [&](int h, int i, float u, float v, float2 t) {           // pair (i, i + half)
        const T x = from_f32<T>(u * t.x - v * t.y), z = from_f32<T>(v * t.x + u * t.y);
        T* dst = q + h * hw + dp + i;
        dst[0] = x;
        dst[half] = z;
        if (qa) {
            qa[h * ap + i] = x;
            qa[h * ap + i + half] = z;
        }
    };
    auto pads = [&](int h) {                                                 // columns behind the rotated part are zero
        for (int i = a.sh.rot + lane; i < a.sh.rp; i += 32) q[h * hw + dp + i] = from_f32<T>(0.f);
        if (qa)
            for (int i = a.sh.rot + lane; i < ap - a.sh.rank; i += 32) qa[h * ap + i] = from_f32<T>(0.f);
    };
    if constexpr (kSmallHead) {
        const float2 t = lane < half ? cs[lane] : make_float2(1.f, 0.f);
        for (int h0 = warp; h0 < heads; h0 += 16) {
            float4 x[2];
            float u[2], v[2];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const float* src = pr + (h0 + 8 * k) * hw;
                const bool in = h0 + 8 * k < heads;
                x[k] = in && 4 * lane < dp ? load4(src + 4 * lane) : make_float4(0.f, 0.f, 0.f, 0.f);
                u[k] = in && lane < half ? src[dp + lane] : 0.f;
                v[k] = in && lane < half ? src[dp + half + lane] : 0.f;
            }
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int h = h0 + 8 * k;
                if (h >= heads) break;
                if (4 * lane < dp) store4(q + h * hw + 4 * lane, x[k]);
                if (lane < half) rotated(h, lane, u[k], v[k], t);
                pads(h);
            }
        }
    } else {
        for (int h = warp; h < heads; h += 8) {
            const float* src = pr + h * hw;
            for (int c = 4 * lane; c < dp; c += 128) store4(q + h * hw + c, load4(src + c));
            for (int i = lane; i < half; i += 32) rotated(h, i, src[dp + i], src[dp + i + half], cs[i]);
            pads(h);
        }
    }
}

// The cache row of a token: normed latent, rotated key part, zeros.
template <typename T>
__device__ __forceinline__ void latent_append(const LatentPreArgs& a, int row, int slot, int pos, const float* __restrict__ y, float* s_part) {
    const int tid = threadIdx.x, rank = a.sh.rank, half = a.sh.rot / 2;
    const int cap = a.cache.capacity[slot];
    if (pos >= cap) {
        if (tid == 0) atomicExch(a.cache.error, 2);                          // page not reserved: skip the write
        return;
    }
    const int page = a.cache.block_table[slot * a.cache.max_pages_per_seq + pos / kPageTokens];
    float ss = 0.f;
    for (int c = tid; c < rank; c += 256) ss += y[c] * y[c];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((tid & 31) == 0) s_part[tid >> 5] = ss;
    __syncthreads();
    ss = ((s_part[0] + s_part[1]) + (s_part[2] + s_part[3])) + ((s_part[4] + s_part[5]) + (s_part[6] + s_part[7]));
    const float rms = sqrtf(ss / (float)rank + a.sh.eps);
    T* __restrict__ dst = static_cast<T*>(a.cache.rows) + ((size_t)page * kPageTokens + pos % kPageTokens) * a.cache.pitch;
    for (int c = tid; c < rank; c += 256) dst[c] = from_f32<T>(y[c] / rms * a.c_norm[c]);
    for (int i = tid; i < half; i += 256) {
        const float u = y[rank + i], v = y[rank + half + i];
        const float2 t = a.cs[(size_t)row * half + i];
        dst[rank + i] = from_f32<T>(u * t.x - v * t.y);
        dst[rank + half + i] = from_f32<T>(v * t.x + u * t.y);
    }
    for (int c = rank + a.sh.rot + tid; c < a.cache.pitch; c += 256) dst[c] = from_f32<T>(0.f);
}

// grid (rows, 2 with latents of its own, else 1), block 256: queries, append.  A stream with little arithmetic: what counts
// is how many loads are under way, hence the register bound.
template <typename T, bool kSmallHead>
__global__ void __launch_bounds__(256, 6)
latent_pre_kernel(const LatentPreArgs a) {
    __shared__ float s_part[8];
    pdl_enter();
    const int row = blockIdx.x, slot = a.row_slot[row];
    if (slot < 0 || slot >= a.cache.max_seqs) return;
    const float* pr = a.proj + (size_t)row * a.sh.pitch();
    if (blockIdx.y == 0) latent_queries<T, kSmallHead>(a, row, pr);
    else latent_append<T>(a, row, slot, a.row_pos[row], pr + a.sh.q_cols(), s_part);
}

int launch_latent_pre(ElemType t, const LatentPreArgs& a, int rows, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
const bool small = a.sh.dp <= 128 && a.sh.rot <= 64;
        launch_pdl(small ? latent_pre_kernel<T, true> : latent_pre_kernel<T, false>, dim3(rows, a.sh.own ? 2 : 1), dim3(256), 0, s, a);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

// grid (rows, heads), block 128: every warp takes every fourth visible key with an online softmax of its own (lane l holds
// latent columns l, l + 32, ...), the four are joined at the end.  NC = latent columns per lane.
template <int NC, typename T>
__global__ void __launch_bounds__(128)
latent_attn_rows_kernel(const LatentShape sh, const T* __restrict__ qa, LatentView cache, const int* __restrict__ row_slot,
                        const int* __restrict__ row_pos, T* __restrict__ out) {
    extern __shared__ float sm[];
    pdl_enter();
    const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int slot = row_slot[row], pos = row_pos[row];
    T* o = out + ((size_t)row * sh.heads + h) * sh.rank;
    if (slot < 0 || slot >= cache.max_seqs || pos >= cache.capacity[slot]) {
        for (int c = tid; c < sh.rank; c += 128) o[c] = from_f32<T>(0.f);
        return;
    }
    const int kd = sh.rank + sh.rot;
    float* s_q = sm;                              // [kd]
    float* s_acc = sm + round_up(kd, 4);          // [4][rank]
    float* s_ml = s_acc + 4 * sh.rank;            // [4][2]
    const T* q = qa + ((size_t)row * sh.heads + h) * sh.row_pitch();
    for (int c = tid; c < kd; c += 128) s_q[c] = to_f32(q[c]);
    __syncthreads();
    const int first = sh.window > 0 ? max(0, pos - sh.window + 1) : 0;
    float m = -INFINITY, l = 0.f, acc[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i) acc[i] = 0.f;
    for (int j = first + warp; j <= pos; j += 4) {
        const int page = cache.block_table[slot * cache.max_pages_per_seq + j / kPageTokens];
        const T* k = static_cast<const T*>(cache.rows) + ((size_t)page * kPageTokens + j % kPageTokens) * cache.pitch;
        float c[NC], d = 0.f;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const int e = lane + 32 * i;
            c[i] = e < sh.rank ? to_f32(k[e]) : 0.f;
            d += e < sh.rank ? c[i] * s_q[e] : 0.f;
        }
        for (int e = sh.rank + lane; e < kd; e += 32) d += to_f32(k[e]) * s_q[e];
#pragma unroll
        for (int x = 16; x > 0; x >>= 1) d += __shfl_xor_sync(0xffffffffu, d, x);
        d *= sh.scale;
        const float mn = fmaxf(m, d), al = expf(m - mn), p = expf(d - mn);
        l = l * al + p;
#pragma unroll
        for (int i = 0; i < NC; ++i) acc[i] = acc[i] * al + p * c[i];
        m = mn;
    }
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const int e = lane + 32 * i;
        if (e < sh.rank) s_acc[warp * sh.rank + e] = acc[i];
    }
    if (lane == 0) { s_ml[2 * warp] = m; s_ml[2 * warp + 1] = l; }
    __syncthreads();
    const float mx = fmaxf(fmaxf(s_ml[0], s_ml[2]), fmaxf(s_ml[4], s_ml[6]));
    float w[4], tot = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) { w[i] = expf(s_ml[2 * i] - mx); tot += w[i] * s_ml[2 * i + 1]; }
    for (int c = tid; c < sh.rank; c += 128)
        o[c] = from_f32<T>((w[0] * s_acc[c] + w[1] * s_acc[sh.rank + c] + w[2] * s_acc[2 * sh.rank + c] + w[3] * s_acc[3 * sh.rank + c]) / tot);
}

int launch_latent_attn_rows(ElemType t, const LatentShape& sh, const void* qa, const LatentView& cache, const int* row_slot,
                            const int* row_pos, int rows, void* out, cudaStream_t s) {
    const size_t smem = (size_t)(round_up(sh.rank + sh.rot, 4) + 4 * sh.rank + 8) * 4;
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        auto go = [&](auto kernel) { launch_pdl(kernel, dim3(rows, sh.heads), dim3(128), smem, s, sh, (const T*)qa, cache, row_slot, row_pos, (T*)out); };
        if (sh.rank <= 64) go(latent_attn_rows_kernel<2, T>);
        else if (sh.rank <= 128) go(latent_attn_rows_kernel<4, T>);
        else if (sh.rank <= 256) go(latent_attn_rows_kernel<8, T>);
        else if (sh.rank <= 512) go(latent_attn_rows_kernel<16, T>);
        else go(latent_attn_rows_kernel<32, T>);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

// Context rows of a pass, cache -> contiguous: latents [ctx][rank], rotated parts [ctx][rp] (zero behind rot).  One warp per row.
__global__ void __launch_bounds__(256)
latent_stage_kernel(int rank, int rot, int rp, LatentView cache, const LatentSpan* __restrict__ spans, __nv_bfloat16* __restrict__ c_stage,
                    __nv_bfloat16* __restrict__ r_stage) {
    const LatentSpan sp = spans[blockIdx.y];
    const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (i >= sp.count) return;
    const int pos = sp.pos0 + i;
    if (pos >= cache.capacity[sp.slot]) return;
    const int page = cache.block_table[sp.slot * cache.max_pages_per_seq + pos / kPageTokens];
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(cache.rows) + ((size_t)page * kPageTokens + pos % kPageTokens) * cache.pitch;
    __nv_bfloat16* c = c_stage + (size_t)(sp.ctx0 + i) * rank;
    __nv_bfloat16* r = r_stage + (size_t)(sp.ctx0 + i) * rp;
    if ((rank & 7) == 0) {
        for (int e = 8 * lane; e < rank; e += 256) *reinterpret_cast<uint4*>(c + e) = *reinterpret_cast<const uint4*>(src + e);
    } else {
        for (int e = lane; e < rank; e += 32) c[e] = src[e];
    }
    for (int e = lane; e < rp; e += 32) r[e] = e < rot ? src[rank + e] : __float2bfloat16_rn(0.f);
}

int launch_latent_stage(const LatentShape& sh, const LatentView& cache, const LatentSpan* d_spans, int n_spans, int max_count, void* c_stage,
                        void* r_stage, cudaStream_t s) {
    latent_stage_kernel<<<dim3(ceil_div(max_count, 8), n_spans), 256, 0, s>>>(sh.rank, sh.rot, sh.rp, cache, d_spans, (__nv_bfloat16*)c_stage,
                                                                             (__nv_bfloat16*)r_stage);
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
