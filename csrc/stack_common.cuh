// Element access and small device helpers of the composed-stack kernels (bf16 or fp32 operands, fp32 arithmetic).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "host_utils.h"

namespace rb {
namespace stack {

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// eight consecutive elements, 16-byte aligned
struct F8 { float v[8]; };
__device__ __forceinline__ F8 unpack8(const uint4& u) {
  F8 r;
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    r.v[2 * i] = __uint_as_float(w[i] << 16);
    r.v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
  return r;
}
__device__ __forceinline__ F8 ld8(const __nv_bfloat16* p) { return unpack8(*reinterpret_cast<const uint4*>(p)); }
__device__ __forceinline__ F8 ld8(const float* p) {
  F8 r;
  *reinterpret_cast<float4*>(r.v) = reinterpret_cast<const float4*>(p)[0];
  *reinterpret_cast<float4*>(r.v + 4) = reinterpret_cast<const float4*>(p)[1];
  return r;
}
__device__ __forceinline__ void st8(float* p, const F8& r) {
  reinterpret_cast<float4*>(p)[0] = *reinterpret_cast<const float4*>(r.v);
  reinterpret_cast<float4*>(p)[1] = *reinterpret_cast<const float4*>(r.v + 4);
}
__device__ __forceinline__ void st8(__nv_bfloat16* p, const F8& r) {
  uint4 u;
  uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 b = __floats2bfloat162_rn(r.v[2 * i], r.v[2 * i + 1]);
    w[i] = *reinterpret_cast<const uint32_t*>(&b);
  }
  *reinterpret_cast<uint4*>(p) = u;
}
template <int V, typename T>
__device__ __forceinline__ void ldv(const T* p, float* v) {
  if constexpr (V == 8) {
    const F8 r = ld8(p);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = r.v[i];
  } else {
    v[0] = ld(p);
  }
}
template <int V, typename T>
__device__ __forceinline__ void stv(T* p, const float* v) {
  if constexpr (V == 8) {
    F8 r;
#pragma unroll
    for (int i = 0; i < 8; ++i) r.v[i] = v[i];
    st8(p, r);
  } else {
    st(p, v[0]);
  }
}

__device__ __forceinline__ float wsum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// 1 / (1 + exp(-x)): IEEE expf and division in 32-bit mode, hardware approximations in 16-bit mode
template <bool kExact>
__device__ __forceinline__ float sigmoid(float x) {
  if constexpr (kExact) return 1.f / (1.f + expf(-x));
  else return __fdividef(1.f, 1.f + __expf(-x));      // x << 0: the denominator overflows to inf, the quotient is 0
}
// the value that an element of type T keeps of x
template <typename T>
__device__ __forceinline__ float round_to(float x) {
  if constexpr (sizeof(T) == 4) return x;
  else return __bfloat162float(__float2bfloat16(x));
}
template <typename T> struct IsExact { static constexpr bool v = sizeof(T) == 4; };

}  // namespace stack
}  // namespace rb
