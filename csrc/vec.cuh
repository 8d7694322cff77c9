// Typed vector access for kernels that run in bf16 (serving) or in true 32-bit: eight elements at a time (one 16-byte
// access for bf16, two for float), converted to and from float registers.
#pragma once
#include "common.cuh"

namespace b2 {

__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }

__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 t = unpack_bf16x2(w[i]);
    f[2 * i] = t.x;
    f[2 * i + 1] = t.y;
  }
}
__device__ __forceinline__ void vload8(const __nv_bfloat16* p, float (&f)[8]) {
  unpack8(*reinterpret_cast<const uint4*>(p), f);
}
__device__ __forceinline__ void vload8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void vstore8(__nv_bfloat16* p, const float (&f)[8]) {
  uint4 u;
  u.x = pack_bf16x2(f[0], f[1]);
  u.y = pack_bf16x2(f[2], f[3]);
  u.z = pack_bf16x2(f[4], f[5]);
  u.w = pack_bf16x2(f[6], f[7]);
  *reinterpret_cast<uint4*>(p) = u;
}
__device__ __forceinline__ void vstore8(float* p, const float (&f)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// Forms for values that are rounded to bf16 next (relative error about 2^-21): one special-function 2^x and one reciprocal.
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + fast_exp2(-1.4426950408889634f * z)); }
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + fast_exp2(-1.4426950408889634f * z)); }
template <typename T>
__device__ __forceinline__ float silu_t(float z) { return sizeof(T) == 2 ? silu_fast(z) : silu_f(z); }
template <typename T>
__device__ __forceinline__ float sigmoid_t(float z) { return sizeof(T) == 2 ? sigmoid_fast(z) : sigmoid_f(z); }

}  // namespace b2

// bf16 / fp32 dispatch of a launcher body: `T` is the activation type inside the braces
#define B2_DISPATCH_T(is_f32, ...)          \
  do {                                      \
    if (is_f32) {                           \
      using T = float;                      \
      __VA_ARGS__                           \
    } else {                                \
      using T = __nv_bfloat16;              \
      __VA_ARGS__                           \
    }                                       \
  } while (0)

#define B2_CHECK_LAUNCH(name)                                        \
  do {                                                               \
    cudaError_t e_ = cudaGetLastError();                             \
    if (e_ != cudaSuccess) {                                         \
      set_error(name " launch failed: %s", cudaGetErrorString(e_));  \
      return 4;                                                      \
    }                                                                \
  } while (0)
