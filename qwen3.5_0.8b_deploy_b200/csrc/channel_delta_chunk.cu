// Chunk-64 prefill of the channel-wise gated delta rule (channel_delta.cu) in two kernels.
//
// With G_t the running sums of the log decays inside a chunk (one per key channel) and S_0 the state at its start:
//     A_ts = beta_t sum_d k_t k_s e^{G_t - G_s}  (s < t),    M_ts = sum_d q_t k_s e^{G_t - G_s}  (s <= t),    T = (I + A)^-1
//     W = T diag(beta) (e^G K),   U' = T diag(beta) V,   U = U' - W S_0
//     O = (e^G Q) S_0 + M U,      S_C = diag(e^{G_C}) S_0 + (e^{G_C - G} K)^T U
// Everything but the lines with S_0 needs no state: the first kernel does it for all chunks at once (convolutions, unit vectors and
// gates included) and leaves W, e^G Q, e^{G_C - G} K, M and U' as images of the shared-memory tiles that the second kernel, which
// walks the chunks of a sequence, multiplies with the state on tcgen05.
//
// A decay is always the product of factors <= 1, never a quotient: pairs of tokens inside a group of four get their factors as
// running products in registers; pairs of groups inside a block of 16, and pairs of blocks, meet on mma.sync with the later
// token decayed from the start of its group (block) and the earlier one decayed up to there, in one copy per later group (block).
// Operands are fp16: unit vectors, decays, beta and T are at most 1, and 11 bits are kept of values.
#include "block_model.cuh"
#include "channel_delta.cuh"
#include "elem.cuh"
#include "tc05.cuh"

#include <algorithm>

namespace b200 {

namespace {
constexpr int kDC = 64;
constexpr uint32_t kTile = kDC * 128;                  // 64 rows of 64 fp16, 128-byte swizzle
constexpr float kDL2e = 1.4426950408889634f;

// An item (chunk and head) of the scratch: W | e^G Q | e^{G_C - G} K (nd tiles each) | M | e^{G_C} | U' per state tile (nv tiles of [64 values][64 tokens])
struct DeltaItem {
    int nd, nv, n_vt;
    __host__ __device__ uint32_t off_k() const { return 2 * nd * kTile; }
    __host__ __device__ uint32_t off_m() const { return 3 * nd * kTile; }
    __host__ __device__ uint32_t off_e() const { return off_m() + kTile; }
    __host__ __device__ uint32_t off_u() const { return off_e() + nd * 256; }
    __host__ __device__ uint32_t bytes() const { return off_u() + n_vt * nv * kTile; }
};
// Items of a sequence start at row0 / 64 + its index: no two sequences meet.
__device__ __forceinline__ size_t first_chunk(int row0, int seq) { return (size_t)(row0 / kDC) + seq; }

__device__ __forceinline__ float ex2c(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcpc(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rsqc(float x) {
    float y;
    asm("rsqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float sigmoidc(float x) { return rcpc(1.0f + ex2c(x * -kDL2e)); }
__device__ __forceinline__ uint32_t sw(int r, int p) { return (uint32_t)(r * 128 + ((p ^ (r & 7)) << 4)); }   // 16-byte piece p of row r
__device__ __forceinline__ float2 unpack_half2(uint32_t v) { return __half22float2(*reinterpret_cast<const __half2*>(&v)); }
__device__ __forceinline__ uint32_t mul_half2(uint32_t a, uint32_t b) {
    const __half2 r = __hmul2(*reinterpret_cast<const __half2*>(&a), *reinterpret_cast<const __half2*>(&b));
    return *reinterpret_cast<const uint32_t*>(&r);
}
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldm2(uint32_t& a, uint32_t& b, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(a), "=r"(b) : "r"(addr));
}

struct DeltaChunkArgs {
    DeltaShape sh;
    DeltaItem item;
    const __nv_bfloat16* qkv;          // [rows][off_b]
    const float* a;                    // [rows][heads * dp] decay pre-activations
    const float* b;                    // [rows][heads]
    const float *conv, *a_log, *dt_bias;   // conv: [4][off_b] for up to four taps, [off_b][taps] for more
    const float* state;
    const LaSeqMeta* seqs;
    int max_seqs;
    unsigned char* scratch;
    int* error;
};

__device__ __forceinline__ float4 unpack4(uint2 v) {
    const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
// Where a pass's inputs of a short convolution are: rows of bf16, and [taps - 1][stride] floats from before the pass.
struct ConvSource {
    const __nv_bfloat16* raw;          // the head's first channel in the pass's first row
    const float* hist;
    int pitch, stride, count, channels, padded;     // channels exist in hist, padded ones in raw
};
// Three rows in front of a pass's first chunk, over what a tile's load brought there: the inputs kept from before, zeros ahead of them.
__device__ __forceinline__ void put_history(unsigned char* tile, int row_bytes, const ConvSource& c, int taps, int tid, int n) {
    for (int i = tid; i < 3 * (row_bytes / 2); i += n) {
        const int r = i / (row_bytes / 2), ch = i % (row_bytes / 2), t = taps - 1 - 3 + r;
        reinterpret_cast<__nv_bfloat16*>(tile)[i] = __float2bfloat16_rn(t >= 0 && ch < c.channels ? c.hist[(size_t)t * c.stride + ch] : 0.f);
    }
}

// Four consecutive tokens x four channels behind a short convolution and silu.  Tokens behind the sequence's end get finite values
// that meet a beta of zero.
// TAPS 4: from a tile of rows tok0 - 3 .. tok0 + 63 (by TMA; the tokens are rows t + 3 .. t + 6), w [4][w_pitch] with leading zeros for fewer taps.
// TAPS 0: any number of taps, from global memory, w [channel][taps].
template <int TAPS>
__device__ __forceinline__ void conv_piece(const unsigned char* tile, int row_bytes, const ConvSource& c, int ch, const float* w, int w_pitch, int taps, int tok0,
                                           int t, float (&o)[4][4]) {
#pragma unroll
    for (int i = 0; i < 4; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    auto add = [&](int i, float4 x, float4 k) { o[i][0] += x.x * k.x; o[i][1] += x.y * k.y; o[i][2] += x.z * k.z; o[i][3] += x.w * k.w; };
    if constexpr (TAPS > 0) {
        float4 wv[TAPS];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wv[j] = load4(w + j * w_pitch);
        const unsigned char* p = tile + t * row_bytes + ch * 2;
#pragma unroll
        for (int r = 0; r < TAPS + 3; ++r) {
            const float4 x = unpack4(*reinterpret_cast<const uint2*>(p + r * row_bytes));
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (r - i >= 0 && r - i < TAPS) add(i, x, wv[r - i]);
        }
    } else {
#pragma unroll 1
        for (int j = 0; j < taps; ++j)
#pragma unroll 1
            for (int i = 0; i < 4; ++i) {
                const int at = tok0 + t + i + j - taps + 1;
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
                if (at >= 0) {
                    if (at < c.count) x = load4(c.raw + (size_t)at * c.pitch + ch);
                } else {
                    const float* h = c.hist + (size_t)(taps - 1 + at) * c.stride + ch;
                    if (ch < c.channels) x.x = h[0];
                    if (ch + 1 < c.channels) x.y = h[1];
                    if (ch + 2 < c.channels) x.z = h[2];
                    if (ch + 3 < c.channels) x.w = h[3];
                }
                const float* wj = w + j;
                const float4 k = make_float4(wj[0], wj[taps], wj[2 * taps], wj[3 * taps]);
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (e == i) add(e, x, k);
            }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] *= sigmoidc(o[i][e]);
}

// Shared memory of the first kernel; rows of K-major tiles are 64 ND + 8 halves apart (an odd number of 16-byte units).
constexpr int kPrepThreads = 512;
constexpr uint32_t kRegion = 17408;                    // 64 rows of 136 halves
constexpr uint32_t kOffKA = 0;                         // staged q, decayed keys (rows), e^G K, then the image of U'
constexpr uint32_t kOffQA = kRegion;                   // staged k, decayed queries (rows), staged v, then the image of W
constexpr uint32_t kOffKB = 2 * kRegion;               // keys decayed to the end of their group, then V
constexpr uint32_t kOffCOL = 3 * kRegion;              // 96 rows of decayed keys (columns), then T diag(beta), a swizzled fp16 tile
constexpr uint32_t kOffAD = kOffCOL + 26112;           // A's diagonal blocks, fp32 [64][kAdP]
constexpr int kAdP = 20;
constexpr uint32_t kOffAT = kOffAD + 64 * kAdP * 4;    // A below them, a swizzled fp16 tile
constexpr uint32_t kOffD = kOffAT + kTile;             // the diagonal blocks' inverses, fp16 [64] rows 48 bytes apart
constexpr uint32_t kOffM = kOffD + 64 * 48;            // image of M
constexpr uint32_t kOffG = kOffM + kTile;              // [17][64 ND] log2 decays up to the start of every group
constexpr uint32_t kOffB = kOffG + 17 * 128 * 4;       // beta [64]
constexpr uint32_t kOffPBar = kOffB + 256;             // loads of q and k, of v; give-up flag
constexpr uint32_t kPrepSmem = kOffPBar + 64;
// T = (I + A)^-1 in blocks of 16.  Threads 0 .. 63 invert the diagonal blocks D_I, a column each by forward substitution in fp32.
__device__ __forceinline__ void invert_blocks(unsigned char* sm, const float* s_beta, int tid) {
    const float* AD = reinterpret_cast<const float*>(sm + kOffAD);
    const int b0 = tid & ~15, col = tid & 15;
    float t[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) t[i] = i == col ? 1.f : 0.f;
#pragma unroll
    for (int i = 1; i < 16; ++i) {
        float acc0 = 0.f, acc1 = 0.f;
#pragma unroll
        for (int j = 0; j < i; j += 4) {
            const float4 a = load4(AD + (b0 + i) * kAdP + j);                 // entries at and above the diagonal are zero
            acc0 += a.x * t[j] + a.z * t[j + 2];
            acc1 += a.y * t[j + 1] + a.w * t[j + 3];
        }
        t[i] -= acc0 + acc1;
    }
    const float beta = s_beta[tid];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        *reinterpret_cast<__half*>(sm + kOffD + (b0 + i) * 48 + col * 2) = __float2half_rn(t[i]);
        *reinterpret_cast<__half*>(sm + kOffCOL + sw(b0 + i, tid >> 3) + 2 * (tid & 7)) = __float2half_rn(t[i] * beta);
    }
}
// A warp per block column J: T_IJ^T = -(sum_K T_KJ^T A_IK^T) D_I^T from top to bottom; a product's accumulators are the next one's A operand.
template <int J>
__device__ __forceinline__ void solve_block_column(unsigned char* sm, uint32_t base, const float* s_beta, int lane) {
    const int g4 = lane >> 2, t4 = lane & 3, r8 = (lane & 7) + ((lane >> 4) & 1) * 8, k8 = (lane >> 3) & 1;
    uint32_t y[4][4];
    ldm4t(y[J], base + kOffD + (16 * J + r8) * 48 + k8 * 16);
    const float b0 = -s_beta[16 * J + g4], b1 = -s_beta[16 * J + g4 + 8];
#pragma unroll
    for (int I = J + 1; I < 4; ++I) {
        float z[2][4] = {}, d[2][4] = {};
        uint32_t b[4];
#pragma unroll
        for (int K = J; K < I; ++K) {
            ldm4(b, base + kOffAT + sw(16 * I + r8, 2 * K + k8));
            mma_16816(z[0], y[K][0], y[K][1], y[K][2], y[K][3], b[0], b[1]);
            mma_16816(z[1], y[K][0], y[K][1], y[K][2], y[K][3], b[2], b[3]);
        }
        const uint32_t a0 = pack_half2(z[0][0], z[0][1]), a1 = pack_half2(z[0][2], z[0][3]), a2 = pack_half2(z[1][0], z[1][1]), a3 = pack_half2(z[1][2], z[1][3]);
        ldm4(b, base + kOffD + (16 * I + r8) * 48 + k8 * 16);
        mma_16816(d[0], a0, a1, a2, a3, b[0], b[1]);
        mma_16816(d[1], a0, a1, a2, a3, b[2], b[3]);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            y[I][2 * j] = pack_half2(-d[j][0], -d[j][1]);
            y[I][2 * j + 1] = pack_half2(-d[j][2], -d[j][3]);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = 16 * I + 8 * j + 2 * t4 + e;
                *reinterpret_cast<__half*>(sm + kOffCOL + sw(t, 2 * J) + 2 * g4) = __float2half_rn(d[j][e] * b0);
                *reinterpret_cast<__half*>(sm + kOffCOL + sw(t, 2 * J + 1) + 2 * g4) = __float2half_rn(d[j][2 + e] * b1);
            }
        }
    }
}
__device__ __forceinline__ void sync_half(int which) { asm volatile("bar.sync %0, 256;" ::"r"(1 + which) : "memory"); }
}  // namespace

// grid (heads, chunks, sequences), block 512, two CTAs per SM.  Thread (tg, c4): tokens 4 tg .. 4 tg + 3, channels 4 c4 .. 4 c4 + 3; with
// more than 64 channels a group of tokens is a warp's.
template <int ND, int TAPS>
__global__ void __launch_bounds__(kPrepThreads, 2)
delta_prep_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, const DeltaChunkArgs A) {
    extern __shared__ __align__(1024) unsigned char sm[];
    constexpr int DK = 64 * ND, LN = 16 * ND, kP = DK + 8;         // channels, lanes per token, row pitch in halves
    const DeltaShape& sh = A.sh;
    const LaSeqMeta sq = A.seqs[blockIdx.z];
    const int h = blockIdx.x, chunk = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
    if (chunk * kDC >= sq.count || sq.slot < 0 || sq.slot >= A.max_seqs) return;
    const uint32_t base = smem_u32(sm);
    float* AD = reinterpret_cast<float*>(sm + kOffAD);
    float* s_g = reinterpret_cast<float*>(sm + kOffG);
    float* s_beta = reinterpret_cast<float*>(sm + kOffB);
    unsigned char* item = A.scratch + ((first_chunk(sq.row0, blockIdx.z) + chunk) * sh.heads + h) * A.item.bytes();
    const int tok0 = chunk * kDC, left = sq.count - tok0, D4 = (sh.dim + 3) / 4 * 4, taps = sh.taps, kvh = h / (sh.heads / sh.kv_heads);
    const __nv_bfloat16* rows = A.qkv + (size_t)sq.row0 * sh.off_b();
    const float* st = A.state + (size_t)sq.slot * sh.state_floats() + (size_t)h * sh.n_vt * sh.tile_floats();
    const float* hist = st + (size_t)sh.dim * sh.vt;
    const ConvSource cq{rows + kvh * sh.dp, hist, sh.off_b(), D4, sq.count, sh.dim, sh.dp};
    const ConvSource ck{rows + sh.off_k() + kvh * sh.dp, hist + (taps - 1) * D4, sh.off_b(), D4, sq.count, sh.dim, sh.dp};
    volatile int* abort_flag = reinterpret_cast<volatile int*>(sm + kOffPBar + 16);
    auto bar = [&](int i) { return base + kOffPBar + 8u * i; };
    if (TAPS > 0 && tid == 480) {
        mbar_init(bar(0), 1);
        mbar_init(bar(1), 1);
        *abort_flag = 0;
        mbar_fence_init();
        fence_proxy_async_smem();
        mbar_arrive_expect_tx(bar(0), 2 * 67 * DK * 2);
        tma_load_2d(base + kOffKA, &map_k, bar(0), kvh * sh.dp, sq.row0 + tok0 - 3);
        tma_load_2d(base + kOffQA, &map_k, bar(0), sh.off_k() + kvh * sh.dp, sq.row0 + tok0 - 3);
    }
    const int tg = tid / LN, c4 = tid % LN, ch = 4 * c4, t0 = 4 * tg;
    const bool act = tg < 16, in = act && ch < sh.dp;               // act: whole warps
    float4 z[4];                                                    // decay pre-activations: requested ahead of the convolutions
    if (in) {
        const float* za = A.a + (size_t)(sq.row0 + tok0) * (sh.heads * sh.dp) + h * sh.dp + ch;
#pragma unroll
        for (int i = 0; i < 4; ++i) z[i] = load4(za + min(t0 + i, left - 1) * (sh.heads * sh.dp));
    }
    if (tid >= 384 && tid < 448) s_beta[tid - 384] = tid - 384 < left ? sigmoidc(A.b[(size_t)(sq.row0 + tok0 + tid - 384) * sh.heads + h]) : 0.f;
    if (tid < 16 * kAdP) reinterpret_cast<float4*>(AD)[tid] = make_float4(0.f, 0.f, 0.f, 0.f);
    reinterpret_cast<uint4*>(sm + kOffM)[tid] = make_uint4(0u, 0u, 0u, 0u);

    uint32_t qh[4][2], kh[4][2];                                    // unit vectors, fp16 pairs
    float g[4][4];                                                  // decays of the four tokens
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        qh[i][0] = qh[i][1] = kh[i][0] = kh[i][1] = 0u;
        g[i][0] = g[i][1] = g[i][2] = g[i][3] = 1.f;
    }
    __syncthreads();
    if constexpr (TAPS > 0) {
        mbar_wait(bar(0), 0, abort_flag);
        if (chunk == 0) {
            put_history(sm + kOffKA, 8 * LN, cq, taps, tid, kPrepThreads);
            put_history(sm + kOffQA, 8 * LN, ck, taps, tid, kPrepThreads);
            __syncthreads();
        }
    }
    if (act) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const int col = n * sh.off_k() + kvh * sh.dp + (in ? ch : 0);
            float o[4][4];
            conv_piece<TAPS>(sm + (n ? kOffQA : kOffKA), 8 * LN, n ? ck : cq, in ? ch : 0, A.conv + col * (TAPS > 0 ? 1 : taps), sh.off_b(), taps, tok0, t0, o);
            float ss[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) ss[i] = in ? (o[i][0] * o[i][0] + o[i][1] * o[i][1]) + (o[i][2] * o[i][2] + o[i][3] * o[i][3]) : 0.f;
#pragma unroll
            for (int x = LN / 2; x > 0; x >>= 1)
#pragma unroll
                for (int i = 0; i < 4; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], x);
            if (in) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float inv = (n ? 1.0f : rsqc((float)sh.dim)) * rsqc(ss[i] + 1e-6f);
                    (n ? kh : qh)[i][0] = pack_half2(o[i][0] * inv, o[i][1] * inv);
                    (n ? kh : qh)[i][1] = pack_half2(o[i][2] * inv, o[i][3] * inv);
                }
            }
        }
        float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
        if (in) {
            const float ea = -expf(A.a_log[h]);
            const float4 d4 = load4(A.dt_bias + h * sh.dp + ch);
            const float dt[4] = {d4.x * kDL2e, d4.y * kDL2e, d4.z * kDL2e, d4.w * kDL2e};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                if (t0 + i >= left) continue;
                const float l0 = ea * delta_softplus2(fmaf(z[i].x, kDL2e, dt[0])), l1 = ea * delta_softplus2(fmaf(z[i].y, kDL2e, dt[1]));
                const float l2 = ea * delta_softplus2(fmaf(z[i].z, kDL2e, dt[2])), l3 = ea * delta_softplus2(fmaf(z[i].w, kDL2e, dt[3]));
                sum = make_float4(sum.x + l0, sum.y + l1, sum.z + l2, sum.w + l3);
                g[i][0] = ex2c(l0); g[i][1] = ex2c(l1); g[i][2] = ex2c(l2); g[i][3] = ex2c(l3);
            }
        }
        store4(s_g + (tg + 1) * DK + ch, sum);
    }
    __syncthreads();
    if (tid < DK) {                                                 // log2 decays from the chunk's start to the start of every group
        float run = 0.f;
        s_g[tid] = 0.f;
#pragma unroll
        for (int j = 1; j <= 16; ++j) { run += s_g[j * DK + tid]; s_g[j * DK + tid] = run; }
        reinterpret_cast<float*>(item + (3 * ND + 1) * kTile)[tid] = ex2c(run);
    }
    if (act) {
        // ---- pairs inside the group: factors are running products ----
        float acc[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) acc[i] = 0.f;
#pragma unroll
        for (int e2 = 0; e2 < 2; ++e2) {
            float2 q[4], k[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { q[i] = unpack_half2(qh[i][e2]); k[i] = unpack_half2(kh[i][e2]); }
#pragma unroll
            for (int s = 0; s < 4; ++s) {
                float wx = k[s].x, wy = k[s].y;                     // key s as token t sees it
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    if (t < s) continue;
                    if (t > s) {
                        wx *= g[t][2 * e2];
                        wy *= g[t][2 * e2 + 1];
                        acc[t * (t - 1) / 2 + s] += k[t].x * wx + k[t].y * wy;
                    }
                    acc[6 + t * (t + 1) / 2 + s] += q[t].x * wx + q[t].y * wy;
                }
            }
        }
        // sixteen sums over the lanes of a token: halve the values while halving the lanes
        int n = 16, at = 0;
#pragma unroll
        for (int x = LN / 2; x > LN / 32; x >>= 1) {
            n >>= 1;
            const bool top = c4 & x;
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                if (e >= n) continue;
                const float y = __shfl_xor_sync(0xffffffffu, top ? acc[e] : acc[e + n], x);
                acc[e] = (top ? acc[e + n] : acc[e]) + y;
            }
            if (top) at += n;
        }
        if constexpr (ND == 2) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 1);
        // pairs (t, s): A: 10 20 21 30 31 32, M: 00 10 11 20 21 22 30 31 32 33, packed as 4 t + s
        const uint32_t codes = at < 8 ? 0x40EDC984u : 0xFEDCA985u;
        const int p = (int)(codes >> (4 * (at & 7))) & 15, t = t0 + (p >> 2), s = t0 + (p & 3);
        if (ND == 1 || !(lane & 1)) {
            if (at < 6) AD[t * kAdP + (s & 15)] = s_beta[t] * acc[0];
            else *reinterpret_cast<__half*>(sm + kOffM + sw(t, s >> 3) + 2 * (s & 7)) = __float2half_rn(acc[0]);
        }
    }
    __syncthreads();
    const float* r0 = s_g + tg * DK + ch;                           // up to this group's start / end, up to the chunk's end
    const float *r1 = r0 + DK, *rC = s_g + 16 * DK + ch;
    auto piece = [&](uint32_t off, int row) { return reinterpret_cast<uint2*>(sm + off + row * kP * 2 + ch * 2); };
    // image of a [64][64 ND] tile, row t0 + i (i < 4), this thread's channels: sw() with t0 a multiple of four
    unsigned char* img = item + (ch >> 6) * kTile + t0 * 128 + (ch & 4) * 2;
    const int pb = ((ch >> 3) & 7) ^ (t0 & 4);
    auto image = [&](uint32_t off, int i) { return reinterpret_cast<uint2*>(img + (off + i * 128 + ((pb ^ i) << 4))); };
    auto scaled = [](uint2 v, uint2 f) { return make_uint2(mul_half2(v.x, f.x), mul_half2(v.y, f.y)); };
    auto factors = [](const float* to, const float* from) {         // 2^(to - from)
        const float4 a = load4(to), b = load4(from);
        return make_uint2(pack_half2(ex2c(a.x - b.x), ex2c(a.y - b.y)), pack_half2(ex2c(a.z - b.z), ex2c(a.w - b.w)));
    };
    const int blk = tg >> 2, own = tg & 3;
    if (act) {
        {
            float run[4] = {1.f, 1.f, 1.f, 1.f};
            const uint2 x = factors(r0, s_g + ch);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
#pragma unroll
                for (int e = 0; e < 4; ++e) run[e] *= g[i][e];
                const uint2 f = make_uint2(pack_half2(run[0], run[1]), pack_half2(run[2], run[3]));
                const uint2 q = scaled(make_uint2(qh[i][0], qh[i][1]), f);
                *piece(kOffQA, t0 + i) = q;
                *piece(kOffKA, t0 + i) = scaled(make_uint2(kh[i][0], kh[i][1]), f);
                *image(ND * kTile, i) = scaled(q, x);
            }
        }
        {
            float run[4] = {1.f, 1.f, 1.f, 1.f};
            const uint2 x = factors(rC, r1);
#pragma unroll
            for (int i = 3; i >= 0; --i) {
                const uint2 k = scaled(make_uint2(kh[i][0], kh[i][1]), make_uint2(pack_half2(run[0], run[1]), pack_half2(run[2], run[3])));
                *piece(kOffKB, t0 + i) = k;
                *image(2 * ND * kTile, i) = scaled(k, x);
#pragma unroll
                for (int e = 0; e < 4; ++e) run[e] *= g[i][e];
            }
        }
        // copies for the later groups of the block: 24 rows per block, 4 + 8 + 12
#pragma unroll 1
        for (int i = own + 1; i < 4; ++i) {
            const uint2 f = factors(s_g + (4 * blk + i) * DK + ch, r1);
            const int row = 24 * blk + (i == 1 ? 0 : i == 2 ? 4 : 12) + 4 * own;
#pragma unroll
            for (int s = 0; s < 4; ++s) *piece(kOffCOL, row + s) = scaled(*piece(kOffKB, t0 + s), f);
        }
    }
    __syncthreads();
    auto a_addr = [&](uint32_t off, int row) { return base + off + ((row + (lane & 15)) * kP + (lane >> 4) * 8) * 2; };
    auto b_addr = [&](uint32_t off, int row) { return base + off + ((row + (lane & 7)) * kP + ((lane >> 3) & 1) * 8) * 2; };
    auto put2 = [&](uint32_t off, int t, int s, float x, float y) {  // entries (t, s), (t, s + 1) of a swizzled tile
        *reinterpret_cast<uint32_t*>(sm + off + sw(t, s >> 3) + 2 * (s & 7)) = pack_half2(x, y);
    };
    auto put_group = [&](bool q, int t, int s, float x, float y) {   // of M or a diagonal block of A
        if (q) put2(kOffM, t, s, x, y);
        else *reinterpret_cast<float2*>(AD + t * kAdP + (s & 15)) = make_float2(s_beta[t] * x, s_beta[t] * y);
    };
    auto product = [&](uint32_t aa, uint32_t ba, float (&d)[4]) {   // 16 rows x 8 columns over all channels
        d[0] = d[1] = d[2] = d[3] = 0.f;
#pragma unroll
        for (int k = 0; k < 4 * ND; ++k) {
            uint32_t a[4], b0, b1;
            ldm4(a, aa + k * 32);
            ldm2(b0, b1, ba + k * 32);
            mma_16816(d, a[0], a[1], a[2], a[3], b0, b1);
        }
    };
#pragma unroll 1
    for (int u = warp; u < 24; u += 16) {   // ---- groups against groups: a block's 16 rows x 8 of its 24 columns at a time ----
        const bool q = u & 1;
        const int b = (u >> 1) & 3, n = u >> 3;
        float d[4];
        product(a_addr(q ? kOffQA : kOffKA, 16 * b), b_addr(kOffCOL, 24 * b + 8 * n), d);
        const int c = 8 * n + 2 * t4, i = c < 4 ? 1 : c < 12 ? 2 : 3, s = 16 * b + c - (i == 1 ? 0 : i == 2 ? 4 : 12);
        if ((g4 >> 2) == i) put_group(q, 16 * b + g4, s, d[0], d[1]);
        if (((g4 + 8) >> 2) == i) put_group(q, 16 * b + g4 + 8, s, d[2], d[3]);
    }
    __syncthreads();
    if (act) {
        // ---- rows decay on from the start of their block, columns up to the start of a later one: 16 + 32 + 48 rows ----
        const uint2 f = factors(r0, s_g + 4 * blk * DK + ch);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            *piece(kOffQA, t0 + i) = scaled(*piece(kOffQA, t0 + i), f);
            *piece(kOffKA, t0 + i) = scaled(*piece(kOffKA, t0 + i), f);
        }
#pragma unroll 1
        for (int I = blk + 1; I < 4; ++I) {
            const uint2 x = factors(s_g + 4 * I * DK + ch, r1);
            const int row = (I == 1 ? 0 : I == 2 ? 16 : 48) + t0;
#pragma unroll
            for (int s = 0; s < 4; ++s) *piece(kOffCOL, row + s) = scaled(*piece(kOffKB, t0 + s), x);
        }
    }
    __syncthreads();
#pragma unroll 1
    for (int u = warp; u < 24; u += 16) {   // ---- blocks against blocks ----
        const bool q = u & 1;
        const int v = u >> 1, I = v < 2 ? 1 : v < 6 ? 2 : 3, n = v - (I == 1 ? 0 : I == 2 ? 2 : 6);
        float d[4];
        product(a_addr(q ? kOffQA : kOffKA, 16 * I), b_addr(kOffCOL, (I == 1 ? 0 : I == 2 ? 16 : 48) + 8 * n), d);
        const float f0 = q ? 1.f : s_beta[16 * I + g4], f1 = q ? 1.f : s_beta[16 * I + g4 + 8];
        put2(q ? kOffM : kOffAT, 16 * I + g4, 8 * n + 2 * t4, d[0] * f0, d[1] * f0);
        put2(q ? kOffM : kOffAT, 16 * I + g4 + 8, 8 * n + 2 * t4, d[2] * f1, d[3] * f1);
    }
    fence_proxy_async_smem();
    __syncthreads();
    const int nv = A.item.nv, kVP = 64 * nv + 8;                    // row pitch of V
    auto fetch_values = [&](int tile) {                             // one thread: the inputs of a state tile's values, over the queries
        mbar_arrive_expect_tx(bar(1), 67 * 128 * nv);
        tma_load_2d(base + kOffQA, &map_v, bar(1), sh.off_v() + h * sh.vp + tile * kMlstmTile, sq.row0 + tok0 - 3);
    };
    auto load_values = [&](int tile, int vt, int n, int which) {    // .. behind their convolution to KB; threads vt of n (which >= 0: half `which` of the CTA)
        const float* hv = hist + tile * sh.tile_floats() + 2 * (taps - 1) * D4;
        const int c0 = tile * kMlstmTile, left_v = sh.vp - c0;
        const ConvSource c{rows + sh.off_v() + h * sh.vp + c0, hv, sh.off_b(), sh.vt, sq.count, sh.vdim - c0, left_v};
        if constexpr (TAPS > 0) {
            mbar_wait(bar(1), tile & 1, abort_flag);
            if (chunk == 0) {
                put_history(sm + kOffQA, 128 * nv, c, taps, vt, n);
                if (which < 0) __syncthreads(); else sync_half(which);
            }
        }
        for (int i = vt; i < 256 * nv; i += n) {
            const int t = 4 * (i >> (nv + 3)), vc = 4 * (i & (16 * nv - 1));
            uint2 r[4] = {};
            if (vc < left_v) {
                float o[4][4];
                conv_piece<TAPS>(sm + kOffQA, 128 * nv, c, vc, A.conv + (sh.off_v() + h * sh.vp + c0 + vc) * (TAPS > 0 ? 1 : taps), sh.off_b(), taps, tok0, t, o);
#pragma unroll
                for (int e = 0; e < 4; ++e) r[e] = make_uint2(pack_half2(o[e][0], o[e][1]), pack_half2(o[e][2], o[e][3]));
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) *reinterpret_cast<uint2*>(sm + kOffKB + ((t + e) * kVP + vc) * 2) = r[e];
        }
    };
    if (warp < 8) {   // ---- T = (I + A)^-1, over the column copies ----
        if (tid < 64) invert_blocks(sm, s_beta, tid);
        sync_half(0);
        if (warp == 0) solve_block_column<0>(sm, base, s_beta, lane);
        else if (warp == 1) solve_block_column<1>(sm, base, s_beta, lane);
        else if (warp == 2) solve_block_column<2>(sm, base, s_beta, lane);
    } else {          // ---- meanwhile M goes out and the first values come in ----
        if (tid == 256) {
            if constexpr (TAPS > 0) fetch_values(0);
            bulk_s2g(item + 3 * ND * kTile, base + kOffM, kTile);
            bulk_commit_group();
        }
        load_values(0, tid - 256, 256, 1);
    }
    if (act) {        // the keys decay from the chunk's start
        const uint2 f = factors(s_g + 4 * blk * DK + ch, s_g + ch);
#pragma unroll
        for (int i = 0; i < 4; ++i) *piece(kOffKA, t0 + i) = scaled(*piece(kOffKA, t0 + i), f);
    }
    __syncthreads();
    {   // ---- W = (T diag(beta)) (e^G K): 16 rows x 16 ND columns per warp ----
        const int i = warp >> 2, c0 = (warp & 3) * 16 * ND;
        float d[2 * ND][4];
#pragma unroll
        for (int n = 0; n < 2 * ND; ++n) d[n][0] = d[n][1] = d[n][2] = d[n][3] = 0.f;
        for (int k = 0; k <= i; ++k) {
            uint32_t a[4];
            ldm4(a, base + kOffCOL + sw(16 * i + (lane & 15), 2 * k + (lane >> 4)));
            const uint32_t ka = base + kOffKA + ((16 * k + (lane & 15)) * kP + c0 + (lane >> 4) * 8) * 2;
#pragma unroll
            for (int n = 0; n < 2 * ND; n += 2) {
                uint32_t b[4];
                ldm4t(b, ka + n * 16);
                mma_16816(d[n], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_16816(d[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
#pragma unroll
        for (int n = 0; n < 2 * ND; ++n) {
            const int c = c0 + 8 * n;
            unsigned char* w = sm + kOffQA + (c >> 6) * kTile;
            *reinterpret_cast<uint32_t*>(w + sw(16 * i + g4, (c >> 3) & 7) + 4 * t4) = pack_half2(d[n][0], d[n][1]);
            *reinterpret_cast<uint32_t*>(w + sw(16 * i + g4 + 8, (c >> 3) & 7) + 4 * t4) = pack_half2(d[n][2], d[n][3]);
        }
    }
    fence_proxy_async_smem();
    __syncthreads();
    if (tid == 0) {
        bulk_s2g(item, base + kOffQA, ND * kTile);
        bulk_commit_group();
    }
    // ---- U'^T = V^T (T diag(beta))^T of every state tile: 16 values x every second (fourth) token tile per warp ----
    for (int tile = 0;; ++tile) {
        const int mt = warp & (4 * nv - 1), part = warp >> (nv + 1), parts = 4 / nv;
        uint32_t a[4][4];
#pragma unroll
        for (int k = 0; k < 4; ++k)
            ldm4t(a[k], base + kOffKB + ((16 * k + (lane & 7) + ((lane >> 4) & 1) * 8) * kVP + 16 * mt + ((lane >> 3) & 1) * 8) * 2);
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            if ((n & (parts - 1)) != part) continue;
            float d[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int k = 0; k <= n >> 1; ++k) {
                uint32_t b0, b1;
                ldm2(b0, b1, base + kOffCOL + sw(8 * n + (lane & 7), 2 * k + ((lane >> 3) & 1)));
                mma_16816(d, a[k][0], a[k][1], a[k][2], a[k][3], b0, b1);
            }
            *reinterpret_cast<uint32_t*>(sm + kOffKA + sw(16 * mt + g4, n) + 4 * t4) = pack_half2(d[0], d[1]);
            *reinterpret_cast<uint32_t*>(sm + kOffKA + sw(16 * mt + g4 + 8, n) + 4 * t4) = pack_half2(d[2], d[3]);
        }
        fence_proxy_async_smem();
        __syncthreads();
        if (tid == 0) {
            bulk_s2g(item + A.item.off_u() + tile * nv * kTile, base + kOffKA, nv * kTile);
            bulk_commit_group();
        }
        if (tile + 1 == sh.n_vt) break;
        if (tid == 0) {                // W and this tile's U' have left their places
            bulk_wait_group_read0();
            if constexpr (TAPS > 0) fetch_values(tile + 1);
        }
        load_values(tile + 1, tid, kPrepThreads, -1);
        __syncthreads();
    }
    if (tid == 0 || tid == 256) bulk_wait_group_read0();            // shared memory may go
    if (TAPS > 0 && tid == 0 && *abort_flag) atomicExch(A.error, 11);
}

// ---- the walk over a sequence's chunks -----------------------------------------------------------------------------------------------
namespace {
constexpr int kWalkThreads = 288;                      // 8 compute warps, copies + MMA issuer
constexpr uint32_t kOffWQ = 0;                         // W | e^G Q
constexpr uint32_t kOffWK = 4 * kTile;                 // e^{G_C - G} K | M
constexpr uint32_t kOffWS = 7 * kTile;                 // S_0^T [128 values][64 ND]
constexpr uint32_t kOffWU = 11 * kTile;                // U^T [128 values][64 tokens]
constexpr uint32_t kOffWE = 13 * kTile;                // e^{G_C}
constexpr uint32_t kOffWBar = kOffWE + 512;
constexpr uint32_t kWalkSmem = kOffWBar + 128;
enum { W_WQ = 0, W_KM, W_B2, W_C2, W_B3, W_C3, W_BARS };
}  // namespace

// grid (heads * state tiles, sequences), two CTAs per SM.  TMEM: S^T (lane = value, up to 128 columns), X = S_0^T W^T, O^T.
template <int ND, int NV>
__global__ void __launch_bounds__(kWalkThreads, 2)
delta_walk_kernel(const DeltaShape sh, const DeltaItem it, const __nv_bfloat16* __restrict__ qkv, const LaSeqMeta* __restrict__ seqs, int max_seqs,
                  const unsigned char* __restrict__ scratch, float* __restrict__ state, float* __restrict__ core, int* __restrict__ error_word) {
    extern __shared__ __align__(1024) unsigned char sm[];
    const uint32_t base = smem_u32(sm);
    if (base & 1023u) {            // the 128-byte swizzle needs 1024-byte aligned tiles
        if (threadIdx.x == 0) atomicExch(error_word, 8);
        return;
    }
    uint64_t* bars = reinterpret_cast<uint64_t*>(sm + kOffWBar);
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + W_BARS);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    auto bar = [&](int i) { return base + kOffWBar + 8u * i; };
    const int h = blockIdx.x / sh.n_vt, tile = blockIdx.x % sh.n_vt, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const LaSeqMeta sq = seqs[blockIdx.y];
    const int n_chunks = (sq.count + kDC - 1) / kDC;
    if (n_chunks <= 0 || sq.slot < 0 || sq.slot >= max_seqs) return;
    if (*reinterpret_cast<volatile int*>(error_word) != 0) return;   // an earlier CTA gave up: do not queue more bounded waits
    float* Sg = state + (size_t)sq.slot * sh.state_floats() + (size_t)(h * sh.n_vt + tile) * sh.tile_floats();
    const unsigned char* item0 = scratch + (first_chunk(sq.row0, blockIdx.y) * sh.heads + h) * it.bytes();
    const size_t step = (size_t)sh.heads * it.bytes();

    if (tid == 0) {
        for (int i = 0; i < W_BARS; ++i) mbar_init(bar(i), (i == W_B2 || i == W_B3) ? 256 : 1);
        *abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 8) {
        tmem_alloc(smem_u32(tmem_slot), 256);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot, tm_s = tmem, tm_x = tmem + 128, tm_o = tmem + 192;

    if (warp == 8) {
        // ------------------------------ copies + MMA issuer ------------------------------
        if (lane == 0) {
            constexpr uint32_t id64 = umma_idesc(kFmtF16, 128, 64, 0, 0);
            constexpr uint32_t id_u = umma_idesc(kFmtF16, 128, 64 * ND, 0, 1);      // B MN-major
            auto load_wq = [&](int c) {
                mbar_arrive_expect_tx(bar(W_WQ), 2 * ND * kTile + ND * 256);
                bulk_g2s(base + kOffWQ, item0 + c * step, 2 * ND * kTile, bar(W_WQ));
                bulk_g2s(base + kOffWE, item0 + c * step + it.off_e(), ND * 256, bar(W_WQ));
            };
            auto load_km = [&](int c) {
                mbar_arrive_expect_tx(bar(W_KM), (ND + 1) * kTile);
                bulk_g2s(base + kOffWK, item0 + c * step + it.off_k(), (ND + 1) * kTile, bar(W_KM));
            };
            load_wq(0);
            load_km(0);
            for (int c = 0; c < n_chunks; ++c) {
                const uint32_t par = c & 1;
                if (!mbar_wait(bar(W_WQ), par, abort_flag)) break;
                if (!mbar_wait(bar(W_B2), par, abort_flag)) break;
                tc_fence_after();
#pragma unroll
                for (int ks = 0; ks < 4 * ND; ++ks) {          // X = S_0^T W^T,  O^T = S_0^T (e^G Q)^T
                    const uint64_t a = umma_smem_desc(base + kOffWS + (ks >> 2) * 2 * kTile + (ks & 3) * 32, 16, 1024);
                    const uint32_t off = (ks >> 2) * kTile + (ks & 3) * 32;
                    umma_f16(tm_x, a, umma_smem_desc(base + kOffWQ + off, 16, 1024), id64, ks > 0 ? 1u : 0u);
                    umma_f16(tm_o, a, umma_smem_desc(base + kOffWQ + ND * kTile + off, 16, 1024), id64, ks > 0 ? 1u : 0u);
                }
                umma_commit(bar(W_C2));
                if (c + 1 < n_chunks) {
                    if (!mbar_wait(bar(W_C2), par, abort_flag)) break;
                    load_wq(c + 1);
                }
                if (!mbar_wait(bar(W_KM), par, abort_flag)) break;
                if (!mbar_wait(bar(W_B3), par, abort_flag)) break;
                tc_fence_after();
#pragma unroll
                for (int ks = 0; ks < 4; ++ks) {               // O^T += U^T M^T,  S^T += U^T (e^{G_C - G} K)
                    const uint64_t a = umma_smem_desc(base + kOffWU + ks * 32, 16, 1024);
                    umma_f16(tm_o, a, umma_smem_desc(base + kOffWK + ND * kTile + ks * 32, 16, 1024), id64, 1u);
                    umma_f16(tm_s, a, umma_smem_desc(base + kOffWK + ks * 2048, kTile, 1024), id_u, 1u);
                }
                umma_commit(bar(W_C3));
                if (c + 1 < n_chunks) {
                    if (!mbar_wait(bar(W_C3), par, abort_flag)) break;
                    load_km(c + 1);
                }
            }
        }
    } else {
        // ------------------------------ compute warps ------------------------------
        const int r = tid & 127, hf = tid >> 7;                // value of S^T, X and O^T; half of the columns
        const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
        const float* s_e = reinterpret_cast<const float*>(sm + kOffWE);
        const int col = tile * kMlstmTile + r;
        bool ok = true;
#pragma unroll 1
        for (int cc = 0; cc < ND; ++cc) {
            const int ch = hf * ND + cc;
            uint32_t sv[32];
#pragma unroll
            for (int e = 0; e < 32; ++e) {
                const int d = ch * 32 + e;
                sv[e] = (d < sh.dim && r < sh.vt) ? __float_as_uint(Sg[(size_t)d * sh.vt + r]) : 0u;
            }
            tmem_st32(tm_s + lane_base + ch * 32, sv);
        }
        tmem_wait_st();
        auto store_out = [&](int c, bool do_store) {           // O^T of chunk c -> core[token][head][value]
            uint32_t ov[32];
            tmem_ld32(tm_o + lane_base + hf * 32, ov);
            tmem_wait_ld();
            if (!do_store || col >= sh.vp || r >= 64 * NV) return;
            const int n_valid = sq.count - c * kDC - hf * 32;
            float* dst = core + (size_t)(sq.row0 + c * kDC + hf * 32) * (sh.heads * sh.vp) + h * sh.vp + col;
#pragma unroll
            for (int j = 0; j < 32; ++j)
                if (j < n_valid) dst[(size_t)j * sh.heads * sh.vp] = __uint_as_float(ov[j]);
        };
        for (int c = 0; c < n_chunks; ++c) {   // after a failed wait the warp keeps the barrier protocol going, without waiting or storing
            const uint32_t par = c & 1;
            uint4 u4[4];                       // U' of this thread's 32 tokens
            if (r < 64 * NV) {
                const unsigned char* u = item0 + c * step + it.off_u() + tile * NV * kTile;
#pragma unroll
                for (int q = 0; q < 4; ++q) u4[q] = __ldcs(reinterpret_cast<const uint4*>(u + sw(r, hf * 4 + q)));
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q) u4[q] = make_uint4(0u, 0u, 0u, 0u);
            }
            if (c > 0) {                       // the previous chunk's last products: its outputs and the state are complete
                if (!mbar_wait_warp(bar(W_C3), (c - 1) & 1, abort_flag)) ok = false;
                tc_fence_after();
            }
            if (!mbar_wait_warp(bar(W_WQ), par, abort_flag)) ok = false;
            // ---- S^T -> fp16 tile, and back decayed to the chunk's end ----
#pragma unroll 1
            for (int cc = 0; cc < ND; ++cc) {
                const int ch = hf * ND + cc;
                uint32_t sv[32];
                tmem_ld32(tm_s + lane_base + ch * 32, sv);
                tmem_wait_ld();
                unsigned char* row = sm + kOffWS + (ch >> 1) * 2 * kTile;
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    uint32_t pk[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) pk[e] = pack_half2(__uint_as_float(sv[q * 8 + 2 * e]), __uint_as_float(sv[q * 8 + 2 * e + 1]));
                    *reinterpret_cast<uint4*>(row + sw(r, (ch & 1) * 4 + q)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                }
#pragma unroll
                for (int e = 0; e < 32; e += 4) {
                    const float4 f = *reinterpret_cast<const float4*>(s_e + ch * 32 + e);
                    sv[e] = __float_as_uint(__uint_as_float(sv[e]) * f.x); sv[e + 1] = __float_as_uint(__uint_as_float(sv[e + 1]) * f.y);
                    sv[e + 2] = __float_as_uint(__uint_as_float(sv[e + 2]) * f.z); sv[e + 3] = __float_as_uint(__uint_as_float(sv[e + 3]) * f.w);
                }
                tmem_st32(tm_s + lane_base + ch * 32, sv);
            }
            if (c > 0) store_out(c - 1, ok);   // ahead of the products that overwrite O^T
            tmem_wait_st();
            fence_proxy_async_smem();
            tc_fence_before();
            mbar_arrive(bar(W_B2));
            // ---- U = U' - W S_0 ----
            if (!mbar_wait_warp(bar(W_C2), par, abort_flag)) ok = false;
            tc_fence_after();
            {
                uint32_t x[32];
                tmem_ld32(tm_x + lane_base + hf * 32, x);
                tmem_wait_ld();
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const uint32_t us[4] = {u4[q].x, u4[q].y, u4[q].z, u4[q].w};
                    uint32_t pk[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float2 f = unpack_half2(us[e]);
                        pk[e] = pack_half2(f.x - __uint_as_float(x[q * 8 + 2 * e]), f.y - __uint_as_float(x[q * 8 + 2 * e + 1]));
                    }
                    *reinterpret_cast<uint4*>(sm + kOffWU + sw(r, hf * 4 + q)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                }
            }
            fence_proxy_async_smem();
            tc_fence_before();
            mbar_arrive(bar(W_B3));
        }
        if (ok && mbar_wait_warp(bar(W_C3), (n_chunks - 1) & 1, abort_flag)) {
            tc_fence_after();
            store_out(n_chunks - 1, true);
#pragma unroll 1
            for (int cc = 0; cc < ND; ++cc) {
                const int ch = hf * ND + cc;
                uint32_t sv[32];
                tmem_ld32(tm_s + lane_base + ch * 32, sv);
                tmem_wait_ld();
#pragma unroll
                for (int e = 0; e < 32; ++e) {
                    const int d = ch * 32 + e;
                    if (d < sh.dim && r < sh.vt) Sg[(size_t)d * sh.vt + r] = __uint_as_float(sv[e]);
                }
            }
            // ---- the convolutions' last inputs: a thread per channel, older tokens first ----
            const int D4 = (sh.dim + 3) / 4 * 4, n = sh.taps - 1, kvh = h / (sh.heads / sh.kv_heads), pitch = sh.off_b();
            float* hist = Sg + (size_t)sh.dim * sh.vt;
            auto keep = [&](float* hs, int stride, int c) {
                for (int j = 0; j < n; ++j) {
                    const int t = sq.count - n + j;
                    hs[(size_t)j * stride] = t >= 0 ? __bfloat162float(qkv[(size_t)(sq.row0 + t) * pitch + c]) : hs[(size_t)(n + t) * stride];
                }
            };
            for (int d = tid; d < sh.dim; d += 256) {
                keep(hist + d, D4, kvh * sh.dp + d);
                keep(hist + n * D4 + d, D4, sh.off_k() + kvh * sh.dp + d);
            }
            for (int v = tid; v < sh.vt; v += 256)
                if (tile * kMlstmTile + v < sh.vdim) keep(hist + 2 * n * D4 + v, sh.vt, sh.off_v() + h * sh.vp + tile * kMlstmTile + v);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 8) {
        tc_fence_after();
        tmem_dealloc(tmem, 256);
    }
    if (tid == 0 && *abort_flag) atomicExch(error_word, 10);
}

static DeltaItem delta_item(const DeltaShape& sh) { return DeltaItem{ceil_div(sh.dim, 64), sh.vt > 64 ? 2 : 1, sh.n_vt}; }

bool delta_chunk_fits(const DeltaShape& sh) { return sh.dim <= 128 && sh.off_b() >= 128; }     // the loads' boxes are up to 128 columns wide

size_t delta_chunk_bytes(const DeltaShape& sh) { return (size_t)sh.heads * delta_item(sh).bytes(); }

int launch_delta_chunk(const DeltaShape& sh, const void* qkv, const float* a, const float* b, const float* conv, const float* a_log, const float* dt_bias,
                       const LaSeqMeta* d_seqs, int n_seqs, int max_count, int rows, int max_seqs, float* state, void* scratch, float* core, int* d_error,
                       cudaStream_t s) {
    const DeltaItem it = delta_item(sh);
    static PerDeviceOnce once;
    B2_PER_DEVICE_ONCE(once,
        for (auto k : {delta_prep_kernel<1, 4>, delta_prep_kernel<2, 4>, delta_prep_kernel<1, 0>, delta_prep_kernel<2, 0>})
            B2_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, kPrepSmem));
        for (auto k : {delta_walk_kernel<1, 1>, delta_walk_kernel<1, 2>, delta_walk_kernel<2, 1>, delta_walk_kernel<2, 2>})
            B2_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, kWalkSmem)));
    const DeltaChunkArgs A{sh, it, (const __nv_bfloat16*)qkv, a, b, conv, a_log, dt_bias, state, d_seqs, max_seqs, (unsigned char*)scratch, d_error};
    CUtensorMap mk, mv;
    auto map = [&](CUtensorMap* m, int cols) -> int {          // 67 rows: a chunk and three in front of it
        const uint64_t dims[2] = {(uint64_t)sh.off_b(), (uint64_t)rows};
        const uint64_t str[1] = {(uint64_t)sh.off_b() * 2};
        const uint32_t box[2] = {(uint32_t)cols, 67};
        return make_tensor_map(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, qkv, dims, str, box, false);
    };
    B2_TRY(map(&mk, 64 * it.nd));
    B2_TRY(map(&mv, 64 * it.nv));
    const dim3 gp(sh.heads, ceil_div(max_count, kDC), n_seqs);
    auto prep = [&](auto kernel) { kernel<<<gp, kPrepThreads, kPrepSmem, s>>>(mk, mv, A); };
    if (it.nd == 2) { if (sh.taps <= 4) prep(delta_prep_kernel<2, 4>); else prep(delta_prep_kernel<2, 0>); }
    else { if (sh.taps <= 4) prep(delta_prep_kernel<1, 4>); else prep(delta_prep_kernel<1, 0>); }
    B2_LAUNCH_CHECK();
    const dim3 gw(sh.heads * sh.n_vt, n_seqs);
    auto walk = [&](auto kernel) {
        kernel<<<gw, kWalkThreads, kWalkSmem, s>>>(sh, it, (const __nv_bfloat16*)qkv, d_seqs, max_seqs, (const unsigned char*)scratch, state, core, d_error);
    };
    if (it.nd == 2) { if (it.nv == 2) walk(delta_walk_kernel<2, 2>); else walk(delta_walk_kernel<2, 1>); }
    else { if (it.nv == 2) walk(delta_walk_kernel<1, 2>); else walk(delta_walk_kernel<1, 1>); }
    B2_LAUNCH_CHECK();
    return 0;
}

}  // namespace b200
