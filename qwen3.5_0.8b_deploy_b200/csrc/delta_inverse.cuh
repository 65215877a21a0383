// Inverse of a unit lower triangular 64 x 64 matrix in shared memory (fp32), shared by the chunked delta-rule kernels.
#pragma once

#include <cuda_runtime.h>

namespace b200 {

// Row pitch (floats) of the fp32 A and T matrices in shared memory: 68 keeps 16-byte alignment and moves consecutive
// rows by four banks, so a warp's row-per-lane float4 accesses do not collide.
constexpr int kLd = 68;

// Blocked inverse of the unit lower triangular I + A (64 x 64, blocks of 16).  With D_I the inverted diagonal blocks,
//     T_II = D_I,      T_IJ = - sum_{K=J}^{I-1} (D_I A_IK) T_KJ     (I > J).
// scale_blocks forms B_IK = D_I A_IK in place of A_IK (six independent 16 x 16 x 16 products, one warp each); then a
// column of T depends only on the same column of the block rows above it, so solve_column_group lets one warp own NC
// columns of block column J from top to bottom: it never meets another warp and needs one product per block row.

// Threads 0 .. 63, one column of a diagonal block each, by forward substitution.  Entries of A at and above the diagonal are zero.
__device__ __forceinline__ void invert_diagonal(const float* AM, float* TF, int tid) {
    const int b0 = (tid >> 4) * 16, col = tid & 15;
    float t[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) t[i] = (i == col) ? 1.f : 0.f;
#pragma unroll
    for (int i = 1; i < 16; ++i) {
        const float* arow = AM + (b0 + i) * kLd + b0;
        float acc0 = 0.f, acc1 = 0.f;
#pragma unroll
        for (int j4 = 0; 4 * j4 < i; ++j4) {
            const float4 a4 = *reinterpret_cast<const float4*>(arow + 4 * j4);
            acc0 += a4.x * t[4 * j4] + a4.z * t[4 * j4 + 2];
            acc1 += a4.y * t[4 * j4 + 1] + a4.w * t[4 * j4 + 3];
        }
        t[i] -= acc0 + acc1;   // rows <= col keep their start value: A is strictly lower and t[j < col] = 0
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) TF[(b0 + i) * kLd + b0 + col] = t[i];
}

// warp w < 6 takes block (I, K) = (1,0) (2,0) (2,1) (3,0) (3,1) (3,2); lane = (half of the rows, column)
__device__ __forceinline__ void scale_blocks(float* AM, const float* TF, int w, int lane) {
    const int I = (w == 0) ? 1 : (w < 3 ? 2 : 3);
    const int K = (w == 0) ? 0 : (w < 3 ? w - 1 : w - 3);
    const int rh = lane >> 4, col = lane & 15;        // rows rh, rh + 2, ..: the two halves' D rows lie four banks apart
    float a[16];
#pragma unroll
    for (int k = 0; k < 16; ++k) a[k] = AM[(16 * I + k) * kLd + 16 * K + col];
    float o[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const float* drow = TF + (16 * I + 2 * i + rh) * kLd + 16 * I;
        float acc0 = 0.f, acc1 = 0.f;
#pragma unroll
        for (int k4 = 0; k4 < 4; ++k4) {
            const float4 d = *reinterpret_cast<const float4*>(drow + 4 * k4);    // entries above the diagonal are zero
            acc0 += d.x * a[4 * k4] + d.z * a[4 * k4 + 2];
            acc1 += d.y * a[4 * k4 + 1] + d.w * a[4 * k4 + 3];
        }
        o[i] = acc0 + acc1;
    }
    __syncwarp();                 // every lane holds its column of A_IK: the block may be overwritten
#pragma unroll
    for (int i = 0; i < 8; ++i) AM[(16 * I + 2 * i + rh) * kLd + 16 * K + col] = o[i];
}

// Lane (rg, c): rows rg, rg + 32 / NC, .. of a 16-row block (RPL = NC / 2 of them: neighbouring lanes' rows lie four
// banks apart), column c0 + c of block column J.
template <int NC, int J>
__device__ __forceinline__ void solve_column_group(const float* BM, float* TF, int c0, int lane) {
    constexpr int RPL = NC / 2, RS = 32 / NC;
    const int rg = lane / NC, c = lane % NC;
#pragma unroll
    for (int I = J + 1; I < 4; ++I) {
        float p[RPL];
#pragma unroll
        for (int i = 0; i < RPL; ++i) p[i] = 0.f;
#pragma unroll
        for (int K = J; K < I; ++K) {
#pragma unroll
            for (int k4 = 0; k4 < 4; ++k4) {
                float t[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) t[e] = TF[(16 * K + 4 * k4 + e) * kLd + c0 + c];
#pragma unroll
                for (int i = 0; i < RPL; ++i) {
                    const float4 bq = *reinterpret_cast<const float4*>(&BM[(16 * I + rg + RS * i) * kLd + 16 * K + 4 * k4]);
                    p[i] += bq.x * t[0] + bq.y * t[1] + bq.z * t[2] + bq.w * t[3];
                }
            }
        }
#pragma unroll
        for (int i = 0; i < RPL; ++i) TF[(16 * I + rg + RS * i) * kLd + c0 + c] = -p[i];
        __syncwarp();             // the next block row reads these entries from other lanes of this warp
    }
}

// Eight warps, behind scale_blocks and a barrier: every warp takes a group of columns of T and works down its block rows; the four
// leftmost groups of 4 columns have the longest way (six 16 x 16 x 4 products), the others less.
__device__ __forceinline__ void solve_columns(const float* BM, float* TF, int warp, int lane) {
    if (warp < 4) solve_column_group<4, 0>(BM, TF, 4 * warp, lane);
    else if (warp < 6) solve_column_group<8, 1>(BM, TF, 16 + 8 * (warp - 4), lane);
    else solve_column_group<8, 2>(BM, TF, 32 + 8 * (warp - 6), lane);
}

}  // namespace b200
