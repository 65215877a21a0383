// Gate arithmetic of the channel-wise delta rule's kernels (fp32).
#pragma once

#include <cuda_runtime.h>

namespace b200 {

__device__ __forceinline__ float delta_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// The same with the fast exponential and logarithm; a short series where 1 + x would lose x.
__device__ __forceinline__ float delta_softplus_fast(float z) {
    const float x = __expf(-fabsf(z));
    return fmaxf(z, 0.f) + (x < 0.02f ? x * (1.f - x * (0.5f - x * (1.f / 3.f))) : __logf(1.f + x));
}

}  // namespace b200
