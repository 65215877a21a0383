// Gated delta rule with a decay per key channel: the token-serial kernel and the head norm.
//
// q, k and v pass short causal convolutions per channel and silu; q and k become unit vectors per head.  Per head, with decays
// g_t = exp(-e^{A} softplus(a_t + dt)) over the key channels and beta_t = sigmoid(b_t):
//     S <- diag(g_t) S_{t-1},   u_t = beta_t (v_t - S^T k_t),   S_t = S + k_t u_t^T,   o_t = S_t^T q_t / sqrt(dim)
// and a head's outputs are RMS-normed and gated.  The state of a head lies in tiles of up to 128 value columns; every tile has
// its own copy of the convolutions' last inputs, so that CTAs that share a head never read what another one writes.
#include "block_model.cuh"
#include "channel_delta.cuh"
#include "elem.cuh"
#include "ptx_utils.cuh"

#include <algorithm>

namespace b200 {

// grid (sequences, heads, tiles), block 256.  Lane l of every warp owns value columns 4l .. 4l + 3 of the tile, warp w the key
// rows w, w + 8, ...; with dim <= 8 NR a thread's part of the state stays in registers over the whole run of tokens (decode: one
// token), else it is streamed through for every token.  Decode loads its state ahead of the wait on the preceding kernel.
// kSmall (up to 128 key channels and four taps): threads 0 .. 127 hold the q and k channels with their inputs and weights in
// registers, the others the values', and everything a token needs is requested before the first use; else they are in shared memory.
template <int NR, typename T, bool kSmall, bool kFuseNorm>
__global__ void __launch_bounds__(256, NR <= 16 ? 2 : 1)
delta_step_kernel(const DeltaStepArgs a, unsigned long long* stamp) {
    extern __shared__ float sm[];
    const DeltaShape& sh = a.sh;
    const int D = sh.dim, D4 = (D + 3) / 4 * 4, taps = sh.taps, h = blockIdx.y, tile = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int hist_n = (taps - 1) * (2 * D4 + sh.vt);
    float* s_q = sm;
    float* s_k = s_q + D4;
    float* s_g = s_k + D4;
    float* s_v = s_g + D4;                           // [128]
    float* s_red = s_v + kMlstmTile;                 // two of [8][128]
    float* s_x = s_red + 16 * kMlstmTile;            // 32 words
    float* s_hist = s_x + 32;                        // q [taps - 1][D4] | k [taps - 1][D4] | v [taps - 1][vt]
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
    float* hist = S + (size_t)D * sh.vt;
    const int c0 = 4 * lane;
    const bool act = c0 < sh.vt, resident = D <= 8 * NR;
    float4 st[NR];
    if (resident && act) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = warp + 8 * i;
            if (d < D) st[i] = __ldcs(reinterpret_cast<const float4*>(S + (size_t)d * sh.vt + c0));
        }
    }
    const int kvh = h / (sh.heads / sh.kv_heads), v0 = h * sh.vp + tile * kMlstmTile;
    // kSmall: this thread's channels (key channel d, or value column c of the tile), their last three inputs and four weights
    const bool keys = tid < 128;
    const int own = keys ? tid : tid - 128, n_own = keys ? D : min(sh.vt, sh.vdim - tile * kMlstmTile);
    const bool mine_in = own < n_own;
    const int col0 = keys ? kvh * sh.dp + own : sh.off_v() + v0 + own, col1 = sh.off_k() + kvh * sh.dp + own;
    float h0[3] = {0.f, 0.f, 0.f}, h1[3] = {0.f, 0.f, 0.f}, w0[4] = {0.f, 0.f, 0.f, 0.f}, w1[4] = {0.f, 0.f, 0.f, 0.f}, dt = 0.f;
    if constexpr (kSmall) {
        if (mine_in) {
            const float* hs = hist + (keys ? own : 2 * (taps - 1) * D4 + own);
            const int step = keys ? D4 : sh.vt;
#pragma unroll
            for (int j = 0; j < 3; ++j) {
                const int i = j - (4 - taps);
                if (i < 0) continue;
                h0[j] = hs[i * step];
                if (keys) h1[j] = hs[((taps - 1) + i) * D4];
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                w0[j] = a.conv4[j * sh.off_b() + col0];
                if (keys) w1[j] = a.conv4[j * sh.off_b() + col1];
            }
            if (keys) dt = a.dt_bias[h * sh.dp + own];
        }
    } else {
        for (int i = tid; i < hist_n; i += 256) s_hist[i] = hist[i];
    }
    const float ea = expf(a.a_log[h]), qn = 1.0f / sqrtf((float)D);
    pdl_enter();
    stamp_begin(stamp);
    // one channel of a short convolution: its history moves on by one token
    auto conv = [&](float x, const float* w, float* hs, int step) {
        float acc = x * w[taps - 1];
        for (int j = 0; j < taps - 1; ++j) {
            const float old = hs[j * step];
            acc += old * w[j];
            hs[j * step] = j + 2 < taps ? hs[(j + 1) * step] : x;
        }
        return times_sigmoid<float>(acc, acc);
    };
    auto conv4 = [](float x, float (&hs)[3], const float (&w)[4]) {
        const float acc = hs[0] * w[0] + hs[1] * w[1] + hs[2] * w[2] + x * w[3];
        hs[0] = hs[1]; hs[1] = hs[2]; hs[2] = x;
        return times_sigmoid<float>(acc, acc);
    };
    if constexpr (!kSmall) __syncthreads();
    for (int t = 0; t < count; ++t) {
        const size_t row = row0 + t;
        const float* pr = a.proj + row * sh.pitch();
        const float* gt = a.gates + row * sh.gate_cols();
        float ssq = 0.f, ssk = 0.f;
        const float braw = pr[sh.off_b() + h];
        if constexpr (kSmall) {
            const float x0 = mine_in ? pr[col0] : 0.f, x1 = mine_in && keys ? pr[col1] : 0.f, z = mine_in && keys ? gt[h * sh.dp + own] : 0.f;
            const float y0 = conv4(x0, h0, w0);
            if (keys) {
                const float y1 = conv4(x1, h1, w1);
                if (mine_in) {
                    s_q[own] = y0;
                    s_k[own] = y1;
                    s_g[own] = expf(-ea * delta_softplus(z + dt));
                }
                ssq = y0 * y0;
                ssk = y1 * y1;
            } else if (own < sh.vt) {
                s_v[own] = y0;
            }
        } else {
        for (int d = tid; d < D; d += 256) {
            const int cq = kvh * sh.dp + d, ck = sh.off_k() + cq;
            const float z = gt[h * sh.dp + d] + a.dt_bias[h * sh.dp + d];
            const float q = conv(pr[cq], a.conv + (size_t)cq * taps, s_hist + d, D4);
            const float k = conv(pr[ck], a.conv + (size_t)ck * taps, s_hist + (taps - 1) * D4 + d, D4);
            s_q[d] = q;
            s_k[d] = k;
            s_g[d] = expf(-ea * delta_softplus(z));
            ssq += q * q;
            ssk += k * k;
        }
        for (int c = tid; c < sh.vt; c += 256) {
            const int cv = sh.off_v() + v0 + c;
            s_v[c] = tile * kMlstmTile + c < sh.vdim ? conv(pr[cv], a.conv + (size_t)cv * taps, s_hist + 2 * (taps - 1) * D4 + c, sh.vt) : 0.f;
        }
        }
        const float beta = 1.0f / (1.0f + expf(-braw));
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            ssq += __shfl_xor_sync(0xffffffffu, ssq, o);
            ssk += __shfl_xor_sync(0xffffffffu, ssk, o);
        }
        if (lane == 0) { s_x[warp] = ssq; s_x[8 + warp] = ssk; }
        __syncthreads();
        ssq = ((s_x[0] + s_x[1]) + (s_x[2] + s_x[3])) + ((s_x[4] + s_x[5]) + (s_x[6] + s_x[7]));
        ssk = ((s_x[8] + s_x[9]) + (s_x[10] + s_x[11])) + ((s_x[12] + s_x[13]) + (s_x[14] + s_x[15]));
        const float iq = qn / sqrtf(ssq + 1e-6f), ik = 1.0f / sqrtf(ssk + 1e-6f);
        // ---- decay, and what the state predicts for this key ----
        float4 p = make_float4(0.f, 0.f, 0.f, 0.f);
        auto decayed = [&](float4 x, int d) -> float4 {
            const float g = s_g[d], k = s_k[d] * ik;
            x.x *= g; x.y *= g; x.z *= g; x.w *= g;
            p.x += x.x * k; p.y += x.y * k; p.z += x.z * k; p.w += x.w * k;
            return x;
        };
        if (act) {
            if (resident) {
#pragma unroll
                for (int i = 0; i < NR; ++i) {
                    const int d = warp + 8 * i;
                    if (d < D) st[i] = decayed(st[i], d);
                }
            } else {
                for (int d = warp; d < D; d += 8) {
                    float4* x = reinterpret_cast<float4*>(S + (size_t)d * sh.vt + c0);
                    *x = decayed(*x, d);
                }
            }
        }
        *reinterpret_cast<float4*>(s_red + warp * kMlstmTile + c0) = p;
        __syncthreads();
        // ---- write, and read with the query ----
        float4 u = make_float4(0.f, 0.f, 0.f, 0.f), o4 = u;
        if (act) {
            u = *reinterpret_cast<const float4*>(s_v + c0);
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                const float4 x = *reinterpret_cast<const float4*>(s_red + w * kMlstmTile + c0);
                u.x -= x.x; u.y -= x.y; u.z -= x.z; u.w -= x.w;
            }
            u.x *= beta; u.y *= beta; u.z *= beta; u.w *= beta;
            auto written = [&](float4 x, int d) -> float4 {
                const float k = s_k[d] * ik, q = s_q[d] * iq;
                x.x += k * u.x; x.y += k * u.y; x.z += k * u.z; x.w += k * u.w;
                o4.x += x.x * q; o4.y += x.y * q; o4.z += x.z * q; o4.w += x.w * q;
                return x;
            };
            if (resident) {
#pragma unroll
                for (int i = 0; i < NR; ++i) {
                    const int d = warp + 8 * i;
                    if (d < D) st[i] = written(st[i], d);
                }
            } else {
                for (int d = warp; d < D; d += 8) {
                    float4* x = reinterpret_cast<float4*>(S + (size_t)d * sh.vt + c0);
                    *x = written(*x, d);
                }
            }
        }
        float* red = s_red + 8 * kMlstmTile;
        *reinterpret_cast<float4*>(red + warp * kMlstmTile + c0) = o4;
        __syncthreads();
        float o = 0.f;
        const int vc = tile * kMlstmTile + tid;
        const bool mine = tid < kMlstmTile && tid < sh.vt && vc < sh.vdim;
        if (mine) {
#pragma unroll
            for (int w = 0; w < 8; ++w) o += red[w * kMlstmTile + tid];
        }
        if constexpr (kFuseNorm) {
            if (tid < kMlstmTile) {
                float ss = o * o;
#pragma unroll
                for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
                if (lane == 0) s_x[16 + warp] = ss;
            }
            __syncthreads();
            if (mine) {
                const float rms = sqrtf(((s_x[16] + s_x[17]) + (s_x[18] + s_x[19])) / (float)sh.vdim + sh.eps);
                const float g = gt[sh.heads * sh.dp + h * sh.vp + vc];
                static_cast<T*>(a.gated)[row * (sh.heads * sh.vp) + h * sh.vp + vc] = from_f32<T>(o / rms * a.norm_w[vc] / (1.0f + expf(-g)));
            } else if (tid < kMlstmTile && vc < sh.vp) {
                static_cast<T*>(a.gated)[row * (sh.heads * sh.vp) + h * sh.vp + vc] = from_f32<T>(0.f);
            }
        } else {
            // padded columns too: the head norm reads whole rows, and the buffer holds what other layers left
            if (tid < kMlstmTile && vc < sh.vp) a.core[row * (sh.heads * sh.vp) + h * sh.vp + vc] = o;
        }
        if (t + 1 < count) __syncthreads();       // what the next token overwrites has been read
    }
    if (resident && act) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = warp + 8 * i;
            if (d < D) __stcs(reinterpret_cast<float4*>(S + (size_t)d * sh.vt + c0), st[i]);
        }
    }
    if constexpr (kSmall) {
        if (mine_in) {
            float* hs = hist + (keys ? own : 2 * (taps - 1) * D4 + own);
            const int step = keys ? D4 : sh.vt;
#pragma unroll
            for (int j = 0; j < 3; ++j) {
                const int i = j - (4 - taps);
                if (i < 0) continue;
                hs[i * step] = h0[j];
                if (keys) hs[((taps - 1) + i) * D4] = h1[j];
            }
        }
        if (stamp) __syncthreads();
    } else {
        __syncthreads();
        for (int i = tid; i < hist_n; i += 256) hist[i] = s_hist[i];
    }
    if (stamp) stamp_end(stamp);
}

int launch_delta_step(ElemType t, const DeltaStepArgs& a, int n, cudaStream_t s) {
    const DeltaShape& sh = a.sh;
    const size_t smem = (3 * (size_t)round_up(sh.dim, 4) + 17 * kMlstmTile + 32 + sh.hist_floats()) * 4;
    const dim3 grid(n, sh.heads, sh.n_vt);
    unsigned long long* stamp = a.seqs ? nullptr : prof_stamp_slot(PROF_DELTA_DECODE);
    int rc = 0;
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        auto go = [&](auto kernel) -> int {
            if (smem > 48 * 1024) B2_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            launch_pdl(kernel, grid, dim3(256), smem, s, a, stamp);
            return 0;
        };
        auto pick = [&](auto fuse) -> int {
            constexpr bool kFuse = decltype(fuse)::value;
            if (sh.dim > 128 || !a.conv4) return sh.dim <= 128 ? go(delta_step_kernel<16, T, false, kFuse>) : go(delta_step_kernel<32, T, false, kFuse>);
            if (sh.dim <= 32) return go(delta_step_kernel<4, T, true, kFuse>);
            if (sh.dim <= 64) return go(delta_step_kernel<8, T, true, kFuse>);
            return go(delta_step_kernel<16, T, true, kFuse>);
        };
        rc = sh.n_vt == 1 ? pick(std::true_type{}) : pick(std::false_type{});
    });
    B2_TRY(rc);
    B2_LAUNCH_CHECK();
    return 0;
}

// A head's outputs over their root mean square, times the weight, times sigmoid(g).  One block per row, a warp per head.
template <typename T, typename G>
__global__ void __launch_bounds__(256)
delta_head_norm_kernel(const float* __restrict__ core, const G* __restrict__ g, int g_pitch, const float* __restrict__ norm_w, float eps, int heads,
                       int vdim, int vp, T* __restrict__ out) {
    pdl_enter();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float* c = core + (size_t)blockIdx.x * heads * vp;
    const G* gr = g + (size_t)blockIdx.x * g_pitch;
    T* o = out + (size_t)blockIdx.x * heads * vp;
    auto gated = [](float4 x, float inv, float4 w, float4 z) {
        return make_float4(times_sigmoid<T>(x.x * inv * w.x, z.x), times_sigmoid<T>(x.y * inv * w.y, z.y), times_sigmoid<T>(x.z * inv * w.z, z.z),
                           times_sigmoid<T>(x.w * inv * w.w, z.w));
    };
    auto rms_inv = [&](float ss) {
#pragma unroll
        for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
        return 1.0f / sqrtf(ss / (float)vdim + eps);
    };
    if (vp <= 128) {                               // two heads' loads under way before the first use
        const int v = 4 * lane;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 w = v < vp ? load4(norm_w + v) : zero;
        for (int h0 = warp; h0 < heads; h0 += 16) {
            float4 x[2], z[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int h = h0 + 8 * i;
                const bool in = h < heads && v < vp;               // columns from vdim on are zero
                x[i] = in ? __ldcs(reinterpret_cast<const float4*>(c + h * vp + v)) : zero;
                z[i] = in ? load4(gr + h * vp + v) : zero;
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int h = h0 + 8 * i;
                const float inv = rms_inv(x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w);
                if (h < heads && v < vp) store4(o + h * vp + v, gated(x[i], inv, w, z[i]));
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
        const float inv = rms_inv(ss);
        for (int v = 4 * lane; v < vp; v += 128) store4(o + h * vp + v, gated(load4(c + h * vp + v), inv, load4(norm_w + v), load4(gr + h * vp + v)));
    }
}

int launch_delta_head_norm(ElemType t, const DeltaShape& sh, const float* core, const void* g, bool g_f32, int g_pitch, const float* norm_w, int rows,
                           void* gated, cudaStream_t s) {
    dispatch_elem(t, [&](auto tag) {
        using T = decltype(tag);
        if (g_f32)
            launch_pdl(delta_head_norm_kernel<T, float>, dim3(rows), dim3(256), 0, s, core, (const float*)g, g_pitch, norm_w, sh.eps, sh.heads, sh.vdim,
                       sh.vp, (T*)gated);
        else
            launch_pdl(delta_head_norm_kernel<T, T>, dim3(rows), dim3(256), 0, s, core, (const T*)g, g_pitch, norm_w, sh.eps, sh.heads, sh.vdim, sh.vp,
                       (T*)gated);
    });
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
