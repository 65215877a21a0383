// Gate arithmetic of the channel-wise delta rule's kernels (fp32).
#pragma once

#include <cuda_runtime.h>

namespace b200 {

__device__ __forceinline__ float delta_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// log2(1 + 2^y) on the special-function unit: softplus in units of ln 2.
__device__ __forceinline__ float delta_softplus2(float y) {
    float x;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(x) : "f"(fminf(y, 100.f)));
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(x) : "f"(1.f + x));
    return y > 24.f ? y : x;
}

}  // namespace b200
