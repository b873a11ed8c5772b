// Storage-type helpers of the mixer kernels: bf16 or fp32 in memory, fp32 in registers.
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

#include "bf16x8.cuh"

namespace l3ci {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename S>
__device__ __forceinline__ S from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// A gate z with its partner u: silu(z) u, or, with a limit, z' sigmoid(alpha z') (u' + 1) of the clamped z' = min(z, limit) and
// u' = clamp(u, -limit, limit).
__device__ __forceinline__ float gated_activation(float z, float u, float limit, float alpha) {
  if (limit > 0.f) {
    z = fminf(z, limit);
    u = fminf(fmaxf(u, -limit), limit) + 1.f;
    return z / (1.f + expf(-alpha * z)) * u;
  }
  return z / (1.f + expf(-z)) * u;
}

// The same to bf16 accuracy (relative error about 1e-6), without the divide's branches.
__device__ __forceinline__ float gated_activation_fast(float z, float u, float limit, float alpha) {
  if (limit > 0.f) {
    z = fminf(z, limit);
    u = fminf(fmaxf(u, -limit), limit) + 1.f;
    return __fdividef(z, 1.f + __expf(-alpha * z)) * u;
  }
  return __fdividef(z, 1.f + __expf(-z)) * u;
}

template <int BYTES>
struct Raw;
template <>
struct Raw<2> { using type = uint16_t; };
template <>
struct Raw<4> { using type = uint32_t; };
template <>
struct Raw<8> { using type = uint2; };
template <>
struct Raw<16> { using type = uint4; };
struct alignas(16) Raw32 { uint4 lo, hi; };
template <>
struct Raw<32> { using type = Raw32; };   // two accesses

template <typename S, int VEC>
__device__ __forceinline__ void load_vec(const S* p, float (&f)[VEC]) {
  union { typename Raw<VEC * sizeof(S)>::type raw; S s[VEC]; } u;
  u.raw = *reinterpret_cast<const typename Raw<VEC * sizeof(S)>::type*>(p);
#pragma unroll
  for (int i = 0; i < VEC; ++i) f[i] = to_f32(u.s[i]);
}
template <typename S, int VEC>
__device__ __forceinline__ void store_vec(S* p, const float (&f)[VEC]) {
  union { typename Raw<VEC * sizeof(S)>::type raw; S s[VEC]; } u;
#pragma unroll
  for (int i = 0; i < VEC; ++i) u.s[i] = from_f32<S>(f[i]);
  *reinterpret_cast<typename Raw<VEC * sizeof(S)>::type*>(p) = u.raw;
}

}  // namespace l3ci
