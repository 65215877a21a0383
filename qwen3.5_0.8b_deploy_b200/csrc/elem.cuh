// Element-type helpers of the kernels that run in bf16 or fp32: conversions, four-element accesses, host dispatch.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "common.cuh"

namespace b200 {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float2 unpack_bf16x2(uint32_t v) {
    return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
}
// v = hi + lo with both terms bf16: about 16 significant bits.
__device__ __forceinline__ void split_bf16x2(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16x2(a, b);
    const float2 h = unpack_bf16x2(hi);
    lo = pack_bf16x2(a - h.x, b - h.y);
}

// Four consecutive elements at an address aligned to four elements.
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(r.x), b = unpack_bf16x2(r.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// x * sigmoid(z): library functions for fp32 outputs, the fast exponential and divide where the result is rounded to bf16.
template <typename T> __device__ __forceinline__ float times_sigmoid(float x, float z);
template <> __device__ __forceinline__ float times_sigmoid<float>(float x, float z) { return x / (1.0f + expf(-z)); }
template <> __device__ __forceinline__ float times_sigmoid<__nv_bfloat16>(float x, float z) { return __fdividef(x, 1.0f + __expf(-z)); }

template <typename F>
inline void dispatch_elem(ElemType t, F&& f) {
    if (t == ELEM_F32) f(float{});
    else f(__nv_bfloat16{});
}

}  // namespace b200
