// Element access for kernels that come in a bf16 and an f32 form: N consecutive elements to and from f32 registers with
// one vector access (N = 1, 2, 4; the address is aligned to the vector).
#pragma once
#include <cuda_bf16.h>
#include "b2/ptx.cuh"

namespace b2 {

template <int N>
__device__ __forceinline__ void load_f32(const float* p, float (&v)[N]) {
  if constexpr (N == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else if constexpr (N == 2) {
    const float2 t = *reinterpret_cast<const float2*>(p);
    v[0] = t.x; v[1] = t.y;
  } else {
    v[0] = *p;
  }
}
template <int N>
__device__ __forceinline__ void load_f32(const __nv_bfloat16* p, float (&v)[N]) {
  if constexpr (N == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    v[0] = ptx::bf16_lo(t.x); v[1] = ptx::bf16_hi(t.x); v[2] = ptx::bf16_lo(t.y); v[3] = ptx::bf16_hi(t.y);
  } else if constexpr (N == 2) {
    const uint32_t t = *reinterpret_cast<const uint32_t*>(p);
    v[0] = ptx::bf16_lo(t); v[1] = ptx::bf16_hi(t);
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int N>
__device__ __forceinline__ void store_f32(float* p, const float (&v)[N]) {
  if constexpr (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else if constexpr (N == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  else *p = v[0];
}
template <int N>
__device__ __forceinline__ void store_f32(__nv_bfloat16* p, const float (&v)[N]) {
  if constexpr (N == 4) *reinterpret_cast<uint2*>(p) = make_uint2(ptx::pack_bf16x2(v[0], v[1]), ptx::pack_bf16x2(v[2], v[3]));
  else if constexpr (N == 2) *reinterpret_cast<uint32_t*>(p) = ptx::pack_bf16x2(v[0], v[1]);
  else *p = __float2bfloat16(v[0]);
}

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
// The same by the special-function unit: log(1 + e^x), for small t = e^-|x| by the series of log1p, which keeps the relative
// precision of slow decays.
__device__ __forceinline__ float softplus_fast(float x) {
  const float t = ptx::ex2(-fabsf(x) * ptx::kLog2e);
  float s = fmaf(t, -1.0f / 8, 1.0f / 7);
  s = fmaf(t, s, -1.0f / 6);
  s = fmaf(t, s, 1.0f / 5);
  s = fmaf(t, s, -1.0f / 4);
  s = fmaf(t, s, 1.0f / 3);
  s = fmaf(t, s, -1.0f / 2);
  s = fmaf(t * t, s, t);
  return fmaxf(x, 0.0f) + (t < 0.125f ? s : ptx::lg2(1.0f + t) * ptx::kLn2);
}
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

}  // namespace b2
