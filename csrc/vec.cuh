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

// eight elements that wait in registers as they came from memory
template <typename T>
struct Packed8 {
  uint4 w[sizeof(T) / 2];
  __device__ __forceinline__ void load(const T* p) {
#pragma unroll
    for (int i = 0; i < static_cast<int>(sizeof(T)) / 2; ++i) w[i] = reinterpret_cast<const uint4*>(p)[i];
  }
  __device__ __forceinline__ void zero() {
#pragma unroll
    for (int i = 0; i < static_cast<int>(sizeof(T)) / 2; ++i) w[i] = make_uint4(0, 0, 0, 0);
  }
  __device__ __forceinline__ void get(float (&f)[8]) const { vload8(reinterpret_cast<const T*>(w), f); }
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// Forms for values that are rounded to bf16 next (relative error about 2^-21): one special-function 2^x and one reciprocal.
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + fast_exp2(-1.4426950408889634f * z)); }
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + fast_exp2(-1.4426950408889634f * z)); }
// silu of two values with one reciprocal between them: 1 / (a b) gives 1 / a and 1 / b.  The exponent is bounded so that
// the product stays finite; past the bound the result is below 1e-17.
__device__ __forceinline__ void silu_pair_fast(float& x, float& y) {
  const float a = 1.f + fast_exp2(fminf(-1.4426950408889634f * x, 62.f)), b = 1.f + fast_exp2(fminf(-1.4426950408889634f * y, 62.f));
  const float r = __fdividef(1.f, a * b);
  x *= r * b;
  y *= r * a;
}
template <typename T>
__device__ __forceinline__ float silu_t(float z) { return sizeof(T) == 2 ? silu_fast(z) : silu_f(z); }
template <typename T>
__device__ __forceinline__ float sigmoid_t(float z) { return sizeof(T) == 2 ? sigmoid_fast(z) : sigmoid_f(z); }

// gelu in its tanh form: 0.5 z (1 + tanh(u)) = z sigmoid(2 u), u = sqrt(2 / pi) (z + 0.044715 z^3)
template <typename T>
__device__ __forceinline__ float gelu_tanh_t(float z) {
  const float u = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
  return z * sigmoid_t<T>(2.f * u);
}

// two fp32 multiplications or fused multiply-adds in one instruction
__device__ __forceinline__ float2 mul_f32x2(float2 a, float2 b) {
  unsigned long long d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)));
  return reinterpret_cast<float2&>(d);
}
__device__ __forceinline__ float2 fma_f32x2(float2 a, float2 b, float2 c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(d)
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)), "l"(reinterpret_cast<unsigned long long&>(c)));
  return reinterpret_cast<float2&>(d);
}

// cap * tanh(z) for a score s = cap * z pressed softly into (-cap, cap).  Near zero: the Taylor series of tanh (relative error
// below 1e-7 for |z| <= SOFTCAP_SERIES); elsewhere 1 - 2 / (1 + e^{2 z}), whose absolute error is a rounding of 1.
constexpr float SOFTCAP_SERIES = 0.4f;
__device__ __forceinline__ float tanh_series(float z) {
  const float t = z * z;
  float r = fmaf(t, 21844.f / 6081075.f, -1382.f / 155925.f);
  r = fmaf(t, r, 62.f / 2835.f);
  r = fmaf(t, r, -17.f / 315.f);
  r = fmaf(t, r, 2.f / 15.f);
  r = fmaf(t, r, -1.f / 3.f);
  return fmaf(z * t, r, z);
}
__device__ __forceinline__ float tanh_wide(float z) {
  return 1.f - 2.f * __fdividef(1.f, 1.f + fast_exp2(fminf(2.f * 1.4426950408889634f * z, 126.f)));
}
template <typename T>
__device__ __forceinline__ float softcap_t(float s, float cap) {
  const float z = s / cap;
  if (sizeof(T) == 4) return cap * tanhf(z);
  return cap * (fabsf(z) <= SOFTCAP_SERIES ? tanh_series(z) : tanh_wide(z));
}

// Weight of the second map of differential attention: exp(lq1 . lk1) - exp(lq2 . lk2) + init, by a whole warp.
// lam: [4, ld] = lq1, lk1, lq2, lk2, zero past the head size.
template <typename T>
__device__ __forceinline__ float diff_lambda(const T* lam, int ld, float init) {
  float a = 0.f, b = 0.f;
  for (int c = threadIdx.x & 31; c < ld; c += 32) {
    a = fmaf(to_f(lam[c]), to_f(lam[ld + c]), a);
    b = fmaf(to_f(lam[2 * ld + c]), to_f(lam[3 * ld + c]), b);
  }
  return expf(warp_sum(a)) - expf(warp_sum(b)) + init;
}

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
