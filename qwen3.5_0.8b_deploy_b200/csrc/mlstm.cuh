// Gate arithmetic of the mLSTM kernels (fp32).
#pragma once

#include <cuda_runtime.h>

namespace b200 {

__device__ __forceinline__ float mlstm_log_input(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float mlstm_log_forget(float z, float cap) {
    const float x = cap * tanhf(z / cap);
    return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

}  // namespace b200
