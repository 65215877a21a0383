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

// One block of 256 threads per row.  The new latents' values are requested before the queries are worked on.
template <typename T>
__global__ void __launch_bounds__(256)
latent_pre_kernel(const LatentPreArgs a) {
    constexpr int kOwn = 4;                    // latent values a thread keeps (ranks of up to 1024)
    __shared__ float s_part[8];
    extern __shared__ float2 s_cs[];
    pdl_enter();
    const LatentShape& sh = a.sh;
    const int row = blockIdx.x, tid = threadIdx.x, half = sh.rot / 2;
    const int slot = a.row_slot[row], pos = a.row_pos[row];
    if (slot < 0 || slot >= a.cache.max_seqs) return;
    const float* pr = a.proj + (size_t)row * sh.pitch();
    const float* y = pr + sh.q_cols();
    float own[kOwn], ss = 0.f;
    if (sh.own) {
#pragma unroll
        for (int k = 0; k < kOwn; ++k) {
            const int c = tid + 256 * k;
            own[k] = c < sh.rank ? y[c] : 0.f;
            ss += own[k] * own[k];
        }
    }
    for (int i = tid; i < half; i += 256) s_cs[i] = a.cs[(size_t)row * half + i];
    const int hw = sh.dp + sh.rp, per = hw / 4;
    T* q = static_cast<T*>(a.q) + (size_t)row * sh.heads * hw;
    // unrotated parts: four columns at a time (hw and dp are multiples of 8)
    const int n4 = sh.heads * per;
#pragma unroll 4
    for (int e = tid; e < n4; e += 256) {
        const int h = e / per, c = 4 * (e - h * per);
        if (c < sh.dp) store4(q + 4 * (size_t)e, load4(pr + 4 * (size_t)e));
    }
    __syncthreads();
    // rotated parts, a pair (i, i + half) at a time; the padded columns behind are zero
    for (int e = tid; e < sh.heads * half; e += 256) {
        const int h = e / half, i = e - h * half;
        const float* src = pr + h * hw + sh.dp;
        const float u = src[i], v = src[i + half];
        const float2 cs = s_cs[i];
        const T ru = from_f32<T>(u * cs.x - v * cs.y), rv = from_f32<T>(v * cs.x + u * cs.y);
        T* dst = q + h * hw + sh.dp;
        dst[i] = ru;
        dst[i + half] = rv;
        if (a.qa) {
            T* qa = static_cast<T*>(a.qa) + ((size_t)row * sh.heads + h) * sh.row_pitch() + sh.rank;
            qa[i] = ru;
            qa[i + half] = rv;
        }
    }
    if (sh.rp > sh.rot) {
        const int pad = sh.rp - sh.rot;
        for (int e = tid; e < sh.heads * pad; e += 256) q[(e / pad) * hw + sh.dp + sh.rot + e % pad] = from_f32<T>(0.f);
    }
    if (a.qa) {                                                    // zero tail behind the rotated part
        const int tail0 = sh.rank + sh.rot, tail = sh.row_pitch() - tail0;
        T* qa = static_cast<T*>(a.qa) + (size_t)row * sh.heads * sh.row_pitch() + tail0;
        for (int e = tid; e < sh.heads * tail; e += 256) qa[(e / tail) * sh.row_pitch() + e % tail] = from_f32<T>(0.f);
    }
    if (!sh.own) return;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((tid & 31) == 0) s_part[tid >> 5] = ss;
    __syncthreads();
    ss = ((s_part[0] + s_part[1]) + (s_part[2] + s_part[3])) + ((s_part[4] + s_part[5]) + (s_part[6] + s_part[7]));
    const float rms = sqrtf(ss / (float)sh.rank + sh.eps);
    if (pos >= a.cache.capacity[slot]) {
        if (tid == 0) atomicExch(a.cache.error, 2);                // page not reserved: skip the write
        return;
    }
    const int page = a.cache.block_table[slot * a.cache.max_pages_per_seq + pos / kPageTokens];
    T* dst = static_cast<T*>(a.cache.rows) + ((size_t)page * kPageTokens + pos % kPageTokens) * a.cache.pitch;
#pragma unroll
    for (int k = 0; k < kOwn; ++k) {
        const int c = tid + 256 * k;
        if (c < sh.rank) dst[c] = from_f32<T>(own[k] / rms * a.c_norm[c]);
    }
    for (int i = tid; i < half; i += 256) {
        const float u = y[sh.rank + i], v = y[sh.rank + half + i];
        const float2 cs = s_cs[i];
        dst[sh.rank + i] = from_f32<T>(u * cs.x - v * cs.y);
        dst[sh.rank + half + i] = from_f32<T>(v * cs.x + u * cs.y);
    }
    for (int c = sh.rank + sh.rot + tid; c < a.cache.pitch; c += 256) dst[c] = from_f32<T>(0.f);
}

int launch_latent_pre(ElemType t, const LatentPreArgs& a, int rows, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        launch_pdl(latent_pre_kernel<T>, dim3(rows), dim3(256), (size_t)(a.sh.rot / 2 + 1) * sizeof(float2), s, a);
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
