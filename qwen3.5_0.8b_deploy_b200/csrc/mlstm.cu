// Matrix memory: the token-serial recurrence and the norms behind it, with exponential gating (mLSTM) or with one constant
// decay per head (lightning attention: S_t = decay S_{t-1} + k_t v_t^T, o_t = S_t^T q_t, with silu on q, k and v; the
// concatenated heads are normed together).
//
// mLSTM: per head, with log input gate i = cap tanh(. / cap) and log forget gate f = logsigmoid(cap tanh(. / cap)):
//     m_t = max(f_t + m_{t-1}, i_t),   S_t = e^{f_t + m_{t-1} - m_t} S_{t-1} + e^{i_t - m_t} k_t v_t^T,   n_t likewise with k_t
//     o_t = S_t^T q_t / (max(|n_t . q_t|, e^{-m_t}) + 1e-6)
// and all of S, n, m start at zero.  The state of a head lies in tiles of up to 128 value columns, each with a copy of n
// and m of its own, so that CTAs that share a head never read what another one writes.
#include "block_model.cuh"
#include "elem.cuh"
#include "mlstm.cuh"
#include "ptx_utils.cuh"

#include <algorithm>

namespace b200 {

// grid (sequences, heads, tiles), block 256.  Lane l of every warp owns value columns 4l .. 4l+3 of the tile, warp w the
// key rows w, w + 8, ...; with dim <= 8 NR a thread's part of the state stays in registers over the whole run of tokens
// (decode: one token), else it is streamed through for every token.  Decode loads its state ahead of the wait on the
// preceding kernel: the state was last written one step earlier.
template <int NR, typename T, bool kGated, bool kFuseNorm>
__global__ void __launch_bounds__(256)
mlstm_step_kernel(const MlstmStepArgs a, unsigned long long* stamp) {
    extern __shared__ float sm[];
    const MlstmShape& sh = a.sh;
    const int D = sh.dim, h = blockIdx.y, tile = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float* s_q = sm;
    const int D4 = (D + 3) / 4 * 4;
    float* s_k = s_q + D4;
    float* s_n = s_k + D4;
    float* s_red = s_n + D4;                // [8][128]
    float* s_x = s_red + 8 * kMlstmTile;    // 16 words
    int slot, row0 = blockIdx.x, count = 1;
    if (a.seqs) {
        pdl_wait();
        const LaSeqMeta q = a.seqs[blockIdx.x];
        slot = q.slot; row0 = q.row0; count = q.count;
    } else {
        slot = a.d_slots[blockIdx.x];
    }
    if (slot < 0 || slot >= a.max_seqs || count <= 0) { pdl_enter(); return; }
    float* S = a.state + (size_t)slot * sh.state_floats() + (size_t)(h * sh.n_vt + tile) * sh.tile_floats();
    float* gn = S + (size_t)D * sh.vt;
    float* gm = gn + D4;
    const int c0 = 4 * lane, vcol = tile * kMlstmTile + c0;       // column in the tile / in the head
    const bool act = c0 < sh.vt;
    const bool resident = D <= 8 * NR;
    float4 st[NR];
    if (resident && act) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = warp + 8 * i;
            if (d < D) st[i] = __ldcs(reinterpret_cast<const float4*>(S + (size_t)d * sh.vt + c0));
        }
    }
    float m = 0.f;
    if constexpr (kGated) {
        m = *gm;
        for (int d = tid; d < D; d += 256) s_n[d] = gn[d];
    }
    pdl_enter();
    stamp_begin(stamp);
    const float q_scale = kGated ? 1.0f / sqrtf((float)D) : 1.0f;
    auto taken = [](float x) { return kGated ? x : times_sigmoid<float>(x, x); };
    const int V = sh.vdim;
    for (int t = 0; t < count; ++t) {
        const size_t row = row0 + t;
        const float* pr = a.proj + row * sh.pitch();
        for (int d = tid; d < D; d += 256) {
            s_q[d] = taken(pr[sh.off_q() + h * sh.dp + d]) * q_scale;
            s_k[d] = taken(pr[sh.off_k() + h * sh.dp + d]);
        }
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (act && vcol < sh.vp) v = *reinterpret_cast<const float4*>(pr + sh.off_v() + h * sh.vp + vcol);
        v = make_float4(taken(v.x), taken(v.y), taken(v.z), taken(v.w));
        float keep, add = 1.f;
        if constexpr (kGated) {
            const float ig = mlstm_log_input(pr[sh.off_i() + h] + a.bias[h], sh.gate_cap);
            const float fg = mlstm_log_forget(pr[sh.off_f() + h] + a.bias[sh.heads + h], sh.gate_cap);
            const float m_new = fmaxf(fg + m, ig);
            keep = expf(fg + m - m_new);
            add = expf(ig - m_new);
            m = m_new;
        } else {
            keep = a.bias[h];
        }
        __syncthreads();
        float4 num = make_float4(0.f, 0.f, 0.f, 0.f);
        auto row_step = [&](float4 x, int d) -> float4 {
            const float kd = add * s_k[d], qd = s_q[d];
            x.x = keep * x.x + kd * v.x; x.y = keep * x.y + kd * v.y;
            x.z = keep * x.z + kd * v.z; x.w = keep * x.w + kd * v.w;
            num.x += x.x * qd; num.y += x.y * qd; num.z += x.z * qd; num.w += x.w * qd;
            return x;
        };
        if (act) {
            if (resident) {
#pragma unroll
                for (int i = 0; i < NR; ++i) {
                    const int d = warp + 8 * i;
                    if (d < D) st[i] = row_step(st[i], d);
                }
            } else {
                for (int d = warp; d < D; d += 8) {
                    float4* p = reinterpret_cast<float4*>(S + (size_t)d * sh.vt + c0);
                    *p = row_step(*p, d);
                }
            }
        }
        float nq = 0.f;
        if constexpr (kGated) for (int d = tid; d < D; d += 256) {
            const float nn = keep * s_n[d] + add * s_k[d];
            s_n[d] = nn;
            nq += nn * s_q[d];
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) nq += __shfl_xor_sync(0xffffffffu, nq, o);
        if (lane == 0) s_x[warp] = nq;
        *reinterpret_cast<float4*>(s_red + warp * kMlstmTile + c0) = num;
        __syncthreads();
        float o = 0.f;
        const int vc = tile * kMlstmTile + tid;
        const bool mine = tid < kMlstmTile && tid < sh.vt && vc < V;
        if (tid < kMlstmTile) {
            nq = ((s_x[0] + s_x[1]) + (s_x[2] + s_x[3])) + ((s_x[4] + s_x[5]) + (s_x[6] + s_x[7]));
            if (mine) {
#pragma unroll
                for (int w = 0; w < 8; ++w) o += s_red[w * kMlstmTile + tid];
                if constexpr (kGated) o /= fmaxf(fabsf(nq), expf(-m)) + 1e-6f;
            }
        }
        if constexpr (kFuseNorm) {
            if (tid < kMlstmTile) {
                float ss = o * o;
#pragma unroll
                for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
                if (lane == 0) s_x[8 + warp] = ss;
            }
            __syncthreads();
            if (mine) {
                const float rms = sqrtf(((s_x[8] + s_x[9]) + (s_x[10] + s_x[11])) / (float)V + sh.eps);
                const float g = pr[sh.off_g() + h * sh.vp + vc];
                const float r = o / rms * a.norm_w[h * sh.vp + vc] / (1.0f + expf(-g));
                static_cast<T*>(a.gated)[row * (sh.heads * sh.vp) + h * sh.vp + vc] = from_f32<T>(r);
            }
        } else {
            // padded columns too: the head norm reads whole rows, and the buffer holds what other layers left
            if (tid < kMlstmTile && vc < sh.vp) a.core[row * (sh.heads * sh.vp) + h * sh.vp + vc] = o;
        }
        if (t + 1 < count) __syncthreads();       // s_q, s_k and the partial sums are free again
    }
    if (resident && act) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = warp + 8 * i;
            if (d < D) __stcs(reinterpret_cast<float4*>(S + (size_t)d * sh.vt + c0), st[i]);
        }
    }
    if constexpr (kGated) {
        for (int d = tid; d < D; d += 256) gn[d] = s_n[d];
        if (tid == 0) *gm = m;
    }
    if (stamp) { __syncthreads(); stamp_end(stamp); }
}

int launch_mlstm_step(ElemType t, const MlstmStepArgs& a, int n, cudaStream_t s) {
    const MlstmShape& sh = a.sh;
    const size_t smem = (3 * (size_t)round_up(sh.dim, 4) + 8 * kMlstmTile + 16) * 4;
    const dim3 grid(n, sh.heads, sh.n_vt);
    unsigned long long* stamp = a.seqs ? nullptr : prof_stamp_slot(PROF_LA_DECODE);
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        auto go = [&](auto kernel) { launch_pdl(kernel, grid, dim3(256), smem, s, a, stamp); };
        auto pick = [&](auto gated, auto fuse) {
            constexpr bool kGated = decltype(gated)::value, kFuse = decltype(fuse)::value;
            if (sh.dim <= 32) go(mlstm_step_kernel<4, T, kGated, kFuse>);
            else if (sh.dim <= 64) go(mlstm_step_kernel<8, T, kGated, kFuse>);
            else if (sh.dim <= 128) go(mlstm_step_kernel<16, T, kGated, kFuse>);
            else go(mlstm_step_kernel<32, T, kGated, kFuse>);
        };
        if (!sh.gated) pick(std::false_type{}, std::false_type{});
        else if (sh.n_vt == 1) pick(std::true_type{}, std::true_type{});
        else pick(std::true_type{}, std::false_type{});
    });
    B2_LAUNCH_CHECK();
    return 0;
}

// The head's outputs over their root mean square, times the norm weight, times sigmoid(g).  One block per row, a warp takes
// heads w, w + 8, ..; for heads of up to 128 values the loads of kUnits of them are under way before the first use.
template <typename T, typename G>
__global__ void __launch_bounds__(256)
mlstm_head_norm_kernel(const float* __restrict__ core, const G* __restrict__ g, int g_pitch, int off_g, const float* __restrict__ norm_w,
                       float eps, int heads, int vdim, int vp, T* __restrict__ out) {
    constexpr int kUnits = 2;
    pdl_enter();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float* c = core + (size_t)blockIdx.x * heads * vp;
    const G* gr = g + (size_t)blockIdx.x * g_pitch + off_g;
    T* o = out + (size_t)blockIdx.x * heads * vp;
    auto gated = [](float4 x, float inv, float4 w, float4 z) {
        return make_float4(times_sigmoid<T>(x.x * inv * w.x, z.x), times_sigmoid<T>(x.y * inv * w.y, z.y), times_sigmoid<T>(x.z * inv * w.z, z.z),
                           times_sigmoid<T>(x.w * inv * w.w, z.w));
    };
    if (vp <= 128) {
        const int v = 4 * lane;
        for (int h0 = warp; h0 < heads; h0 += 8 * kUnits) {
            float4 x[kUnits], z[kUnits], w[kUnits];
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < kUnits; ++i) {
                const int h = h0 + 8 * i;
                const bool in = h < heads && v < vp;              // columns from vdim on are zero
                x[i] = in ? __ldcs(reinterpret_cast<const float4*>(c + h * vp + v)) : zero;
                z[i] = in ? load4(gr + h * vp + v) : zero;
                w[i] = in ? load4(norm_w + h * vp + v) : zero;
            }
#pragma unroll
            for (int i = 0; i < kUnits; ++i) {
                const int h = h0 + 8 * i;
                float ss = x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
#pragma unroll
                for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
                const float inv = 1.0f / sqrtf(ss / (float)vdim + eps);
                if (h < heads && v < vp) store4(o + h * vp + v, gated(x[i], inv, w[i], z[i]));
            }
        }
        return;
    }
    for (int h = warp; h < heads; h += 8) {
        float ss = 0.f;
        for (int v = 4 * lane; v < vp; v += 128) {
            const float4 x = load4(c + h * vp + v);
            ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
        }
#pragma unroll
        for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
        const float inv = 1.0f / sqrtf(ss / (float)vdim + eps);
        for (int v = 4 * lane; v < vp; v += 128)
            store4(o + h * vp + v, gated(load4(c + h * vp + v), inv, load4(norm_w + h * vp + v), load4(gr + h * vp + v)));
    }
}

int launch_mlstm_head_norm(ElemType t, const MlstmShape& sh, const float* core, const void* g, bool g_f32, int g_pitch, const float* norm_w,
                           int rows, void* gated, cudaStream_t s) {
    const dim3 grid(rows);
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        if (g_f32)
            launch_pdl(mlstm_head_norm_kernel<T, float>, grid, dim3(256), 0, s, core, (const float*)g, g_pitch, sh.off_g(), norm_w, sh.eps, sh.heads,
                       sh.vdim, sh.vp, (T*)gated);
        else
            launch_pdl(mlstm_head_norm_kernel<T, T>, grid, dim3(256), 0, s, core, (const T*)g, g_pitch, sh.off_g(), norm_w, sh.eps, sh.heads, sh.vdim,
                       sh.vp, (T*)gated);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

// All heads of a row over their common root mean square, times the weight, times sigmoid(g).  One block per row; rows of up
// to 4096 values stay in registers between the two passes.  Columns from vdim on in every head are zero.
template <typename T, typename G>
__global__ void __launch_bounds__(256)
row_norm_gate_kernel(const float* __restrict__ core, const G* __restrict__ g, int g_pitch, int off_g, const float* __restrict__ norm_w, float eps,
                     int cols, int n, T* __restrict__ out) {
    __shared__ float s_part[8];
    pdl_enter();
    const float* c = core + (size_t)blockIdx.x * cols;
    const G* gr = g + (size_t)blockIdx.x * g_pitch + off_g;
    T* o = out + (size_t)blockIdx.x * cols;
    auto gated = [](float4 x, float inv, float4 w, float4 z) {
        return make_float4(times_sigmoid<T>(x.x * inv * w.x, z.x), times_sigmoid<T>(x.y * inv * w.y, z.y), times_sigmoid<T>(x.z * inv * w.z, z.z),
                           times_sigmoid<T>(x.w * inv * w.w, z.w));
    };
    auto block_sum = [&](float v) {
#pragma unroll
        for (int k = 16; k > 0; k >>= 1) v += __shfl_xor_sync(0xffffffffu, v, k);
        if ((threadIdx.x & 31) == 0) s_part[threadIdx.x >> 5] = v;
        __syncthreads();
        return ((s_part[0] + s_part[1]) + (s_part[2] + s_part[3])) + ((s_part[4] + s_part[5]) + (s_part[6] + s_part[7]));
    };
    float ss = 0.f;
    if (cols <= 4096) {
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        float4 x[4], z[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int v = 4 * (threadIdx.x + 256 * i);
            x[i] = v < cols ? __ldcs(reinterpret_cast<const float4*>(c + v)) : zero;
            z[i] = v < cols ? load4(gr + v) : zero;
            ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
        }
        const float inv = 1.0f / sqrtf(block_sum(ss) / (float)n + eps);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int v = 4 * (threadIdx.x + 256 * i);
            if (v < cols) store4(o + v, gated(x[i], inv, load4(norm_w + v), z[i]));
        }
        return;
    }
    for (int v = 4 * threadIdx.x; v < cols; v += 1024) {
        const float4 x = load4(c + v);
        ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss) / (float)n + eps);
    for (int v = 4 * threadIdx.x; v < cols; v += 1024) store4(o + v, gated(load4(c + v), inv, load4(norm_w + v), load4(gr + v)));
}

int launch_row_norm_gate(ElemType t, const MlstmShape& sh, const float* core, const void* g, bool g_f32, int g_pitch, const float* norm_w, int rows,
                         void* gated, cudaStream_t s) {
    const int cols = sh.heads * sh.vp, n = sh.heads * sh.vdim;
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        if (g_f32)
            launch_pdl(row_norm_gate_kernel<T, float>, dim3(rows), dim3(256), 0, s, core, (const float*)g, g_pitch, sh.off_g(), norm_w, sh.eps, cols, n,
                       (T*)gated);
        else
            launch_pdl(row_norm_gate_kernel<T, T>, dim3(rows), dim3(256), 0, s, core, (const T*)g, g_pitch, sh.off_g(), norm_w, sh.eps, cols, n, (T*)gated);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

// One block of 256 threads per row.
template <typename T>
__global__ void __launch_bounds__(256)
silu_cols_kernel(T* __restrict__ p, int cols, int pitch) {
    pdl_enter();
    T* r = p + (size_t)blockIdx.x * pitch;
#pragma unroll 4
    for (int c = 4 * threadIdx.x; c < cols; c += 1024) {
        const float4 v = load4(r + c);
        store4(r + c, make_float4(times_sigmoid<T>(v.x, v.x), times_sigmoid<T>(v.y, v.y), times_sigmoid<T>(v.z, v.z), times_sigmoid<T>(v.w, v.w)));
    }
}

int launch_silu_cols(ElemType t, void* p, int rows, int cols, int pitch, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        launch_pdl(silu_cols_kernel<T>, dim3(rows), dim3(256), 0, s, (T*)p, cols, pitch);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
