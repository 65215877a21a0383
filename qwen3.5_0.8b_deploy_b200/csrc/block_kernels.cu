// Element-wise kernels of layer-described models: scaled embedding, RMS norm on a sublayer's output with the residual add,
// gated products, soft caps, and the row bookkeeping of a pass.  Any width; four values per thread and access where it divides.
#include "block_model.cuh"
#include "elem.cuh"
#include "ptx_utils.cuh"

#include <algorithm>

namespace b200 {

__global__ void row_map_kernel(const LaSeqMeta* __restrict__ seqs, const int* __restrict__ lens, int* __restrict__ row_slot,
                               int* __restrict__ row_pos) {
    const LaSeqMeta q = seqs[blockIdx.y];
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= q.count) return;
    row_slot[q.row0 + i] = q.slot;
    row_pos[q.row0 + i] = (lens ? lens[q.slot] : 0) + i;
}

int launch_row_map(const LaSeqMeta* d_seqs, int n_seqs, int max_count, const int* lens, int* row_slot, int* row_pos, cudaStream_t s) {
    row_map_kernel<<<dim3(ceil_div(max_count, 256), n_seqs), 256, 0, s>>>(d_seqs, lens, row_slot, row_pos);
    B2_LAUNCH_CHECK();
    return 0;
}

// One block of 64 threads per row: cos and sin of position times frequency, the product in double and reduced to one turn.
__global__ void __launch_bounds__(64)
rot_table_kernel(const int* __restrict__ row_pos, const double* __restrict__ freq, int half, float2* __restrict__ table) {
    pdl_enter();
    const double pos = row_pos[blockIdx.x];
    for (int i = threadIdx.x; i < half; i += 64) {
        const double turns = pos * freq[i] * 0.15915494309189535;
        float2 cs;
        sincosf((float)((turns - rint(turns)) * 6.283185307179586), &cs.y, &cs.x);
        table[(size_t)blockIdx.x * half + i] = cs;
    }
}

int launch_rot_table(const int* row_pos, const double* freq, int half, int rows, float2* table, cudaStream_t s) {
    launch_pdl(rot_table_kernel, dim3(rows), dim3(64), 0, s, row_pos, freq, half, table);
    B2_LAUNCH_CHECK();
    return 0;
}

template <typename T>
__global__ void __launch_bounds__(128)
embed_scaled_kernel(const int* __restrict__ tokens, const T* __restrict__ embed, int vocab, int width, float scale,
                    const int* __restrict__ d_slots, const int* __restrict__ lens, int max_seqs, int* __restrict__ row_slot,
                    int* __restrict__ row_pos, float* __restrict__ x, T* __restrict__ xt) {
    pdl_enter();
    const int row = blockIdx.x;
    if (d_slots && threadIdx.x == 0) {
        const int slot = d_slots[row];
        row_slot[row] = slot;
        row_pos[row] = (lens && slot >= 0 && slot < max_seqs) ? lens[slot] : 0;
    }
    const int tok = min(max(tokens[row], 0), vocab - 1);
    const T* e = embed + (size_t)tok * width;
    if ((width & 3) == 0) {
        for (int c = 4 * threadIdx.x; c < width; c += 512) {
            const float4 v = load4(e + c), r = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
            store4(x + (size_t)row * width + c, r);
            store4(xt + (size_t)row * width + c, r);
        }
        return;
    }
    for (int c = threadIdx.x; c < width; c += 128) {
        const float v = to_f32(e[c]) * scale;
        x[(size_t)row * width + c] = v;
        xt[(size_t)row * width + c] = from_f32<T>(v);
    }
}

int launch_embed_scaled(ElemType t, const int* tokens, const void* embed, int vocab, int width, float scale, int rows, const int* d_slots,
                        const int* lens, int max_seqs, int* row_slot, int* row_pos, float* x, void* xt, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        launch_pdl(embed_scaled_kernel<T>, dim3(rows), dim3(128), 0, s, tokens, (const T*)embed, vocab, width, scale, d_slots, lens, max_seqs,
                   row_slot, row_pos, x, (T*)xt);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

__device__ __forceinline__ float block_sum128(float v, float* s_part) {     // blocks of 128 threads
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if ((threadIdx.x & 31) == 0) s_part[threadIdx.x >> 5] = v;
    __syncthreads();
    return (s_part[0] + s_part[1]) + (s_part[2] + s_part[3]);
}

// One block per row.  Rows of up to 2048 values whose width is a multiple of four stay in registers between the two passes.
template <typename T, bool kResidual>
__global__ void __launch_bounds__(128)
norm_rows_kernel(const float* __restrict__ y, const int* __restrict__ row_index, const float* __restrict__ w, float eps, int width,
                 float* __restrict__ x, T* __restrict__ xt) {
    __shared__ float s_part[4];
    pdl_enter();
    const size_t src = (size_t)(row_index ? row_index[blockIdx.x] : blockIdx.x) * width, dst = (size_t)blockIdx.x * width;
    if ((width & 3) == 0 && width <= 2048) {
        float4 v[4];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 4 * (threadIdx.x + 128 * i);
            v[i] = c < width ? *reinterpret_cast<const float4*>(y + src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
        const float rms = sqrtf(block_sum128(ss, s_part) / (float)width + eps);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 4 * (threadIdx.x + 128 * i);
            if (c >= width) break;
            const float4 ww = *reinterpret_cast<const float4*>(w + c);
            float4 r = make_float4(v[i].x / rms * ww.x, v[i].y / rms * ww.y, v[i].z / rms * ww.z, v[i].w / rms * ww.w);
            if constexpr (kResidual) {
                const float4 h = *reinterpret_cast<const float4*>(x + dst + c);
                r = make_float4(h.x + r.x, h.y + r.y, h.z + r.z, h.w + r.w);
                *reinterpret_cast<float4*>(x + dst + c) = r;
            }
            store4(xt + dst + c, r);
        }
        return;
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < width; c += 128) { const float v = y[src + c]; ss += v * v; }
    const float rms = sqrtf(block_sum128(ss, s_part) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += 128) {
        float r = y[src + c] / rms * w[c];
        if constexpr (kResidual) { r += x[dst + c]; x[dst + c] = r; }
        xt[dst + c] = from_f32<T>(r);
    }
}

int launch_post_norm_residual(ElemType t, const float* y, const float* w, float eps, int rows, int width, float* x, void* xt, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        launch_pdl(norm_rows_kernel<T, true>, dim3(rows), dim3(128), 0, s, y, nullptr, w, eps, width, x, (T*)xt);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

int launch_rms_norm_rows(ElemType t, const float* x, const int* row_index, const float* w, float eps, int rows, int width, void* out,
                         cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        launch_pdl(norm_rows_kernel<T, false>, dim3(rows), dim3(128), 0, s, x, row_index, w, eps, width, nullptr, (T*)out);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

// x += add (a repeated pass starts so), out = x / rms * w.  One block per row.
template <typename T, bool kAdd>
__global__ void __launch_bounds__(128)
pre_norm_kernel(float* __restrict__ x, const float* __restrict__ add, const float* __restrict__ w, float eps, int width, T* __restrict__ out) {
    __shared__ float s_part[4];
    pdl_enter();
    const size_t at = (size_t)blockIdx.x * width;
    if ((width & 3) == 0 && width <= 2048) {
        float4 v[4];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 4 * (threadIdx.x + 128 * i);
            v[i] = c < width ? *reinterpret_cast<const float4*>(x + at + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (kAdd && c < width) {
                const float4 e = *reinterpret_cast<const float4*>(add + at + c);
                v[i] = make_float4(v[i].x + e.x, v[i].y + e.y, v[i].z + e.z, v[i].w + e.w);
                *reinterpret_cast<float4*>(x + at + c) = v[i];
            }
            ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
        const float rms = sqrtf(block_sum128(ss, s_part) / (float)width + eps);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 4 * (threadIdx.x + 128 * i);
            if (c >= width) break;
            const float4 ww = *reinterpret_cast<const float4*>(w + c);
            store4(out + at + c, make_float4(v[i].x / rms * ww.x, v[i].y / rms * ww.y, v[i].z / rms * ww.z, v[i].w / rms * ww.w));
        }
        return;
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < width; c += 128) {
        float v = x[at + c];
        if (kAdd) { v += add[at + c]; x[at + c] = v; }
        ss += v * v;
    }
    const float rms = sqrtf(block_sum128(ss, s_part) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += 128) out[at + c] = from_f32<T>(x[at + c] / rms * w[c]);
}

int launch_pre_norm(ElemType t, float* x, const float* add, const float* w, float eps, int rows, int width, void* out, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        launch_pdl(add ? pre_norm_kernel<T, true> : pre_norm_kernel<T, false>, dim3(rows), dim3(128), 0, s, x, add, w, eps, width, (T*)out);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

__global__ void __launch_bounds__(256)
softcap_kernel(float* __restrict__ p, size_t n, float cap) {
    pdl_enter();
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (size_t)gridDim.x * 256) p[i] = cap * tanhf(p[i] / cap);
}

int launch_softcap(float* logits, size_t n, float cap, cudaStream_t s) {
    launch_pdl(softcap_kernel, dim3((unsigned)std::min<size_t>((n + 255) / 256, 148 * 16)), dim3(256), 0, s, logits, n, cap);
    B2_LAUNCH_CHECK();
    return 0;
}

// 0.5 z (1 + tanh y) = z / (1 + e^{-2y}), y = sqrt(2 / pi) (z + 0.044715 z^3)
template <typename T>
__device__ __forceinline__ float gelu_tanh(float z) {
    return times_sigmoid<T>(z, 1.5957691216057308f * (z + 0.044715f * z * z * z));
}

template <typename T, int kAct>
__device__ __forceinline__ float activated(float z) {
    if constexpr (kAct == B200ATTN_ACT_SILU) return times_sigmoid<T>(z, z);
    else return gelu_tanh<T>(z);
}

// Blocks of 128 threads: one per row, or (few rows) several along it.
template <typename T, int kAct>
__global__ void __launch_bounds__(128)
act_mul_kernel(const T* __restrict__ gu, int ff, T* __restrict__ act) {
    pdl_enter();
    const T* g = gu + (size_t)blockIdx.x * 2 * ff;
    T* o = act + (size_t)blockIdx.x * ff;
    if ((ff & 3) == 0) {
#pragma unroll 4
        for (int c = 4 * (threadIdx.x + 128 * blockIdx.y); c < ff; c += 512 * gridDim.y) {
            const float4 a = load4(g + c), u = load4(g + ff + c);
            store4(o + c, make_float4(activated<T, kAct>(a.x) * u.x, activated<T, kAct>(a.y) * u.y, activated<T, kAct>(a.z) * u.z, activated<T, kAct>(a.w) * u.w));
        }
        return;
    }
    for (int c = threadIdx.x + 128 * blockIdx.y; c < ff; c += 128 * gridDim.y) o[c] = from_f32<T>(activated<T, kAct>(to_f32(g[c])) * to_f32(g[ff + c]));
}

int launch_act_mul(ElemType t, int f, const void* gu, int rows, int ff, void* act, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        launch_pdl(f == B200ATTN_ACT_SILU ? act_mul_kernel<T, B200ATTN_ACT_SILU> : act_mul_kernel<T, B200ATTN_ACT_GELU_TANH>, dim3(rows, rows < 1024 ? ceil_div(ff, 512) : 1), dim3(128), 0, s, (const T*)gu, ff, (T*)act);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

__global__ void lens_advance_kernel(int* __restrict__ lens, int n_layers, int max_seqs, const int* __restrict__ d_slots,
                                    const LaSeqMeta* __restrict__ seqs, int n) {
    pdl_enter();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const int slot = seqs ? seqs[i].slot : d_slots[i], count = seqs ? seqs[i].count : 1;
    if (slot < 0 || slot >= max_seqs) return;
    for (int l = 0; l < n_layers; ++l) lens[l * max_seqs + slot] += count;
}

int launch_lens_advance(int* lens, int n_layers, int max_seqs, const int* d_slots, const LaSeqMeta* d_seqs, int n, cudaStream_t s) {
    launch_pdl(lens_advance_kernel, dim3(ceil_div(n, 128)), dim3(128), 0, s, lens, n_layers, max_seqs, d_slots, d_seqs, n);
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
