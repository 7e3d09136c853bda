// Element access that is the same code for the 16-bit storage types and for fp32: scalars and groups of four.
#pragma once
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>

#include "b200/primitives.cuh"

namespace b200 {

__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_float(__half v) { return __half2float(v); }

template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
template <> __device__ __forceinline__ __half from_float<__half>(float v) { return __float2half(v); }

// four consecutive elements (the address is aligned to four elements)
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 load4(const __half* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_f16x2(v.x), b = unpack_f16x2(v.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ void store4(__half* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_f16x2(v.x, v.y), pack_f16x2(v.z, v.w));
}

// Functions of fp32 values on their way into storage of type T: the math library's in the 32-bit mode; with 16-bit storage short
// forms whose error (about 1e-6) is far below a rounding of the result.
template <typename T>
__device__ __forceinline__ float exp_t(float z) { return sizeof(T) == 4 ? expf(z) : __expf(z); }
template <typename T>
__device__ __forceinline__ float silu(float z) { return sizeof(T) == 4 ? z / (1.f + expf(-z)) : __fdividef(z, 1.f + __expf(-z)); }
template <typename T>
__device__ __forceinline__ float inv_sqrt(float z) { return sizeof(T) == 4 ? 1.f / sqrtf(z) : rsqrtf(z); }
template <typename T>
__device__ __forceinline__ float tanh_t(float z) {
  if (sizeof(T) == 4) return tanhf(z);
  const float e = __expf(-2.f * fabsf(z));   // tanh |z| = (1 - e) / (1 + e)
  return copysignf(__fdividef(1.f - e, 1.f + e), z);
}

}  // namespace b200

// Runs `...` with the type alias T bound to the element type of a dtype code (bf16, f16 or f32).
#define B200_DISPATCH_FLOAT(dtype, ...)                                                             \
  do {                                                                                              \
    if ((dtype) == ::b200::kBF16) { using T = __nv_bfloat16; __VA_ARGS__ }                          \
    else if ((dtype) == ::b200::kF16) { using T = __half; __VA_ARGS__ }                             \
    else if ((dtype) == ::b200::kF32) { using T = float; __VA_ARGS__ }                              \
    else return ::b200::set_error(::b200::kErrBadArgument, "dtype %d is not a float type", (dtype)); \
  } while (0)
