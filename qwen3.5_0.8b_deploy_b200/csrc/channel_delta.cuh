// Gate arithmetic of the channel-wise delta rule's kernels (fp32).
#pragma once

#include <cuda_runtime.h>

namespace b200 {

__device__ __forceinline__ float delta_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

}  // namespace b200
