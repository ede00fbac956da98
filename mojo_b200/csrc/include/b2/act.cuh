// Activation functions of matrix-product epilogues, with their constants as parameters (B2EpiAct in b2/api.h).
#pragma once
#include "b2/api.h"
#include "b2/ptx.cuh"

namespace b2 {

constexpr B2EpiAct kPlainAct{INFINITY, 1.0f, 0.0f, 0.0f};

// Gated linear unit g * sigmoid(alpha g) * (u + up_bias) with g <= limit and |u| <= limit; kPlainAct makes it SwiGLU.
__device__ __forceinline__ float glu(const B2EpiAct& a, float g, float u) {
  g = fminf(g, a.limit);
  u = fminf(fmaxf(u, -a.limit), a.limit);
  return g * ptx::rcp(1.0f + ptx::ex2(-g * (ptx::kLog2e * a.alpha))) * (u + a.up_bias);
}
__device__ __forceinline__ float relu2(float x) {
  const float r = fmaxf(x, 0.0f);
  return r * r;
}
__device__ __forceinline__ float softcap(float x, float cap) { return cap * tanhf(x / cap); }

}  // namespace b2
