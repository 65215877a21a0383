// Differential attention: the step behind the input projection (norm, rotation, append), and the attention of any size.
//
// A head has two queries and a key / value head two keys per token (maps); both softmax maps weigh the same values, and the head's
// output is a1 - lambda a2 over its root mean square, times 1 - diff.  Position i sees j <= i with i - j < window or j < keep.
// In a cache page every key / value head has a block of 64 rows [k of map 1 | k of map 2 | v | zeros].
#include "block_model.cuh"
#include "elem.cuh"
#include "ptx_utils.cuh"

namespace b200 {

// One vector of a row (a map of a query or key): RMS norm, rotation of the pairs (2i, 2i + 1), conversion.  A warp per vector;
// vectors of up to 128 values sit in registers, four per lane.
template <typename T>
__device__ __forceinline__ void norm_rotate(const float* __restrict__ src, const float* __restrict__ w, const float2* __restrict__ cs, int dim, int dp,
                                            int half, float eps, T* __restrict__ dst, int lane) {
    float ss = 0.f;
    if (dp <= 128) {
        const int c = 4 * lane;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < dp) x = load4(src + c);                       // padded columns are zero
        ss = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float rms = sqrtf(ss / (float)dim + eps);
        if (c >= dp) return;
        const float4 ww = load4(w + c);                       // [dp], zero behind dim
        x = make_float4(x.x / rms * ww.x, x.y / rms * ww.y, x.z / rms * ww.z, x.w / rms * ww.w);
        if (2 * lane < half) { const float2 t = cs[2 * lane]; const float u = x.x, v = x.y; x.x = u * t.x - v * t.y; x.y = v * t.x + u * t.y; }
        if (2 * lane + 1 < half) { const float2 t = cs[2 * lane + 1]; const float u = x.z, v = x.w; x.z = u * t.x - v * t.y; x.w = v * t.x + u * t.y; }
        store4(dst + c, x);
        return;
    }
    for (int c = lane; c < dim; c += 32) ss += src[c] * src[c];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rms = sqrtf(ss / (float)dim + eps);
    for (int c = 2 * lane; c < dp; c += 64) {
        float u = src[c] / rms * w[c], v = src[c + 1] / rms * w[c + 1];
        if (c / 2 < half) {
            const float2 t = cs[c / 2];
            const float r = u * t.x - v * t.y;
            v = v * t.x + u * t.y;
            u = r;
        }
        dst[c] = from_f32<T>(u);
        dst[c + 1] = from_f32<T>(v);
    }
}

// One block of 256 threads per row; a warp takes every eighth of the row's vectors: queries, keys, values.
template <typename T>
__global__ void __launch_bounds__(256)
diff_pre_kernel(const DiffPreArgs a) {
    pdl_enter();
    const DiffShape& sh = a.sh;
    const int row = blockIdx.x, slot = a.row_slot[row], pos = a.row_pos[row], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (slot < 0 || slot >= a.cache.max_seqs) return;
    const int H = sh.heads, G = sh.kv_heads, dp = sh.dp, hp = sh.hp(), half = sh.rot / 2, per = H / G;
    const float* pr = a.proj + (size_t)row * sh.pitch();
    const float2* cs = a.cs + (size_t)row * half;
    const bool fits = pos < a.cache.capacity[slot];
    if (!fits && threadIdx.x == 0) atomicExch(a.cache.error, 2);             // page not reserved: skip the write
    T* page = nullptr;
    if (fits)
        page = static_cast<T*>(a.cache.rows) + (size_t)a.cache.block_table[slot * a.cache.max_pages_per_seq + pos / kPageTokens] * kPageTokens * sh.row_pitch() +
               (size_t)(pos % kPageTokens) * hp;
    for (int u = warp; u < 2 * H + 3 * G; u += 8) {
        if (u < 2 * H) {
            const int h = u >> 1, map = u & 1;
            T* dst;
            if (a.qd) {
                const int qp = sh.qp();
                dst = static_cast<T*>(a.qd) + (((size_t)row * G + h / per) * 16 + 8 * map + h % per) * qp;
                for (int c = lane; c < dp; c += 32) dst[(1 - map) * dp + c] = from_f32<T>(0.f);
                if (lane < 8) dst[2 * dp + lane] = from_f32<T>(0.f);
                dst += map * dp;
            } else {
                dst = static_cast<T*>(a.q) + ((size_t)row * H * 2 + u) * dp;
            }
            norm_rotate(pr + u * dp, a.q_norm, cs, sh.dim, dp, half, sh.eps, dst, lane);
        } else if (u < 2 * H + 2 * G) {
            const int k = u - 2 * H;
            if (fits) norm_rotate(pr + sh.off_k() + k * dp, a.k_norm, cs, sh.dim, dp, half, sh.eps, page + (size_t)(k >> 1) * kPageTokens * hp + (k & 1) * dp, lane);
        } else if (fits) {
            const int g = u - 2 * H - 2 * G;
            const float* v = pr + sh.off_v() + g * sh.vp;
            T* dst = page + (size_t)g * kPageTokens * hp + 2 * dp;
            for (int c = 4 * lane; c < sh.vp; c += 128) store4(dst + c, load4(v + c));
            if (lane < 8) dst[sh.vp + lane] = from_f32<T>(0.f);
        }
    }
}

// The same for vectors of 4 LPV (64 or 128) columns: LPV lanes per vector, and the loads of all of a warp's first kU rounds of
// vectors are under way before the first use.
template <typename T, int LPV>
__global__ void __launch_bounds__(256)
diff_pre_vec_kernel(const DiffPreArgs a) {
    constexpr int kU = 4, kPer = 8 * (32 / LPV);                // vectors per round of a block
    pdl_enter();
    const DiffShape& sh = a.sh;
    const int row = blockIdx.x, slot = a.row_slot[row], pos = a.row_pos[row];
    if (slot < 0 || slot >= a.cache.max_seqs) return;
    const int H = sh.heads, G = sh.kv_heads, dp = 4 * LPV, hp = sh.hp(), half = sh.rot / 2, per = H / G, n = 2 * (H + G);
    const int first = threadIdx.x / LPV, lane = threadIdx.x % LPV, c = 4 * lane;
    const float* pr = a.proj + (size_t)row * sh.pitch();
    float4 x[kU];
    auto fetch = [&](int v0) {
#pragma unroll
        for (int i = 0; i < kU; ++i) {
            const int v = v0 + i * kPer;                        // queries and keys lie behind one another
            x[i] = v < n ? __ldcs(reinterpret_cast<const float4*>(pr + v * dp + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    };
    fetch(first);
    const float4 wq = load4(a.q_norm + c), wk = load4(a.k_norm + c);     // [dp], zero behind dim
    const float2* cs = a.cs + (size_t)row * half;
    const float2 one = make_float2(1.f, 0.f), t0 = 2 * lane < half ? cs[2 * lane] : one, t1 = 2 * lane + 1 < half ? cs[2 * lane + 1] : one;
    const bool fits = pos < a.cache.capacity[slot];
    if (!fits && threadIdx.x == 0) atomicExch(a.cache.error, 2);         // page not reserved: skip the write
    T* page = nullptr;
    if (fits)
        page = static_cast<T*>(a.cache.rows) + (size_t)a.cache.block_table[slot * a.cache.max_pages_per_seq + pos / kPageTokens] * kPageTokens * sh.row_pitch() +
               (size_t)(pos % kPageTokens) * hp;
    for (int i = threadIdx.x; fits && i < G * sh.vp / 4; i += 256) {     // values
        const int g = 4 * i / sh.vp, cv = 4 * i % sh.vp;
        store4(page + (size_t)g * kPageTokens * hp + 2 * dp + cv, __ldcs(reinterpret_cast<const float4*>(pr + sh.off_v() + 4 * i)));
    }
    if (fits && threadIdx.x < 8 * G) page[(size_t)(threadIdx.x >> 3) * kPageTokens * hp + 2 * dp + sh.vp + (threadIdx.x & 7)] = from_f32<T>(0.f);
    for (int v0 = first; v0 - first < n; v0 += kU * kPer) {              // the same number of rounds in every lane
        if (v0 != first) fetch(v0);
        float ss[kU];
#pragma unroll
        for (int i = 0; i < kU; ++i) ss[i] = (x[i].x * x[i].x + x[i].y * x[i].y) + (x[i].z * x[i].z + x[i].w * x[i].w);
#pragma unroll
        for (int o = LPV / 2; o > 0; o >>= 1)
#pragma unroll
            for (int i = 0; i < kU; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
#pragma unroll
        for (int i = 0; i < kU; ++i) {
            const int v = v0 + i * kPer;
            if (v >= n) break;
            const float inv = 1.0f / sqrtf(ss[i] / (float)sh.dim + sh.eps);
            const float4 w = v < 2 * H ? wq : wk;
            const float4 y = make_float4(x[i].x * inv * w.x, x[i].y * inv * w.y, x[i].z * inv * w.z, x[i].w * inv * w.w);
            const float4 r = make_float4(y.x * t0.x - y.y * t0.y, y.y * t0.x + y.x * t0.y, y.z * t1.x - y.w * t1.y, y.w * t1.x + y.z * t1.y);
            const int hh = v >> 1, map = v & 1;
            if (v >= 2 * H) {
                if (fits) store4(page + (size_t)(hh - H) * kPageTokens * hp + map * dp + c, r);
            } else if (a.qd) {
                const int qp = sh.qp();
                T* dst = static_cast<T*>(a.qd) + (((size_t)row * G + hh / per) * 16 + 8 * map + hh % per) * qp;
                store4(dst + map * dp + c, r);
                store4(dst + (1 - map) * dp + c, make_float4(0.f, 0.f, 0.f, 0.f));
                if (lane < 2) store4(dst + 2 * dp + c, make_float4(0.f, 0.f, 0.f, 0.f));
            } else {
                store4(static_cast<T*>(a.q) + ((size_t)row * H * 2 + v) * dp + c, r);
            }
        }
    }
}

int launch_diff_pre(ElemType t, const DiffPreArgs& a, int rows, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        launch_pdl(a.sh.dp == 64 ? diff_pre_vec_kernel<T, 16> : a.sh.dp == 128 ? diff_pre_vec_kernel<T, 32> : diff_pre_kernel<T>, dim3(rows), dim3(256), 0, s, a);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

// grid (rows, heads), block 256: warps 0 - 3 take map 1, the others map 2; of its map's visible keys a warp takes every fourth with
// an online softmax of its own (lane l holds value columns l, l + 32, ...), the partial results are joined at the end.
template <int NC, typename T>
__global__ void __launch_bounds__(256)
diff_attn_rows_kernel(const DiffShape sh, float lambda, const T* __restrict__ q, LatentView cache, const int* __restrict__ row_slot,
                      const int* __restrict__ row_pos, T* __restrict__ out) {
    extern __shared__ float sm[];
    pdl_enter();
    const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, map = warp >> 2;
    const int slot = row_slot[row], pos = row_pos[row], D = sh.dim, V = sh.vdim, hp = sh.hp();
    T* o = out + ((size_t)row * sh.heads + h) * sh.vp;
    if (slot < 0 || slot >= cache.max_seqs || pos >= cache.capacity[slot]) {
        for (int c = tid; c < sh.vp; c += 256) o[c] = from_f32<T>(0.f);
        return;
    }
    float* s_q = sm;                       // [2][D]
    float* s_acc = s_q + 2 * D;            // [8][V]
    float* s_ml = s_acc + 8 * V;           // [8][2], then the block sum
    const T* qr = q + ((size_t)row * sh.heads + h) * 2 * sh.dp;
    for (int c = tid; c < 2 * D; c += 256) s_q[c] = to_f32(qr[c < D ? c : sh.dp + c - D]);
    __syncthreads();
    const int first = sh.window > 0 ? max(0, pos - sh.window + 1) : 0, kept = min(sh.keep, first), n_keys = kept + pos - first + 1;
    const T* base = static_cast<const T*>(cache.rows) + (size_t)(h / (sh.heads / sh.kv_heads)) * kPageTokens * hp;
    const float* sq = s_q + map * D;
    float m = -INFINITY, l = 0.f, acc[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i) acc[i] = 0.f;
    for (int j = warp & 3; j < n_keys; j += 4) {
        const int key = j < kept ? j : first + (j - kept);
        const int page = cache.block_table[slot * cache.max_pages_per_seq + key / kPageTokens];
        const T* kr = base + (size_t)page * kPageTokens * sh.row_pitch() + (size_t)(key % kPageTokens) * hp;
        float d = 0.f;
        for (int e = lane; e < D; e += 32) d += to_f32(kr[map * sh.dp + e]) * sq[e];
#pragma unroll
        for (int x = 16; x > 0; x >>= 1) d += __shfl_xor_sync(0xffffffffu, d, x);
        d *= sh.scale;
        const float mn = fmaxf(m, d), al = expf(m - mn), p = expf(d - mn);
        l = l * al + p;
        const T* vr = kr + 2 * sh.dp;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const int e = lane + 32 * i;
            acc[i] = acc[i] * al + (e < V ? p * to_f32(vr[e]) : 0.f);
        }
        m = mn;
    }
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const int e = lane + 32 * i;
        if (e < V) s_acc[warp * V + e] = acc[i];
    }
    if (lane == 0) { s_ml[2 * warp] = m; s_ml[2 * warp + 1] = l; }
    __syncthreads();
    float w[2][4], mx[2], tot[2] = {0.f, 0.f};
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const float* ml = s_ml + 8 * k;
        mx[k] = fmaxf(fmaxf(ml[0], ml[2]), fmaxf(ml[4], ml[6]));
#pragma unroll
        for (int i = 0; i < 4; ++i) { w[k][i] = expf(ml[2 * i] - mx[k]); tot[k] += w[k][i] * ml[2 * i + 1]; }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < V; c += 256) {
        float a[2];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float* x = s_acc + 4 * k * V + c;
            a[k] = (w[k][0] * x[0] + w[k][1] * x[V] + w[k][2] * x[2 * V] + w[k][3] * x[3 * V]) / tot[k];
        }
        const float d = a[0] - lambda * a[1];
        s_acc[c] = d;                      // read by this thread only, above and below
        ss += d * d;
    }
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    if (lane == 0) s_ml[warp] = ss;
    __syncthreads();
    ss = ((s_ml[0] + s_ml[1]) + (s_ml[2] + s_ml[3])) + ((s_ml[4] + s_ml[5]) + (s_ml[6] + s_ml[7]));
    const float f = (1.0f - sh.diff) / sqrtf(ss / (float)V + sh.eps);
    for (int c = tid; c < sh.vp; c += 256) o[c] = from_f32<T>(c < V ? s_acc[c] * f : 0.f);
}

int launch_diff_attn_rows(ElemType t, const DiffShape& sh, float lambda, const void* q, const LatentView& cache, const int* row_slot,
                          const int* row_pos, int rows, void* out, cudaStream_t s) {
    const size_t smem = (size_t)(2 * sh.dim + 8 * sh.vdim + 16) * 4;
    int rc = 0;
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        auto go = [&](auto kernel) -> int {
            if (smem > 48 * 1024) B2_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            launch_pdl(kernel, dim3(rows, sh.heads), dim3(256), smem, s, sh, lambda, (const T*)q, cache, row_slot, row_pos, (T*)out);
            return 0;
        };
        if (sh.vdim <= 64) rc = go(diff_attn_rows_kernel<2, T>);
        else if (sh.vdim <= 128) rc = go(diff_attn_rows_kernel<4, T>);
        else if (sh.vdim <= 256) rc = go(diff_attn_rows_kernel<8, T>);
        else rc = go(diff_attn_rows_kernel<32, T>);
    });
    B2_TRY(rc);
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
