// What an attention layer does beyond plain causal softmax: a sliding window or chunks, a soft cap on the scores, a bias by distance,
// a sink, a factor on the result.
#pragma once
#include "b2/api.h"
#include "b2/f32x2.cuh"
#include "b2/ptx.cuh"

namespace b2 {

struct ScoreMods {
  int window;         // positions a row sees, its own included
  int chunk;          // a row sees positions of its own run of `chunk` only; 0: of all
  float cap_log2;     // cap * log2(e); 0: no cap
  float cap_arg;      // scale / cap
  float out_scale;
  const float* bias;  // [2, heads]: r1 and r2 of r1_h ln(1 + r2_h distance), which is taken off a score; null: nothing is
  int heads;
  bool sink;          // the softmax has one more score, zero, without a value

  // The first position that a row at `pos` sees.
  __device__ __forceinline__ int first(int pos) const {
    const int w = max(0, pos - window + 1);
    return chunk > 0 ? max(w, pos - static_cast<int>(static_cast<uint32_t>(pos) % static_cast<uint32_t>(chunk))) : w;
  }
  // log2(e) times the bias of head factors (r1, r2), since ln(z) log2(e) = log2(z).
  __device__ __forceinline__ static float distance(float2 r, int gap) { return r.x * ptx::lg2(fmaf(r.y, static_cast<float>(gap), 1.0f)); }
  __device__ __forceinline__ float2 head_bias(int head) const { return make_float2(bias[head], bias[heads + head]); }

  // log2(e) times the scores of raw dot products: scaled, or capped as cap * tanh(x), x = dot * scale / cap. All lanes of a warp
  // call it together. Where no |x| of the warp exceeds one, tanh(x) = x P(x^2), with P fitted to tanh(x) / x on [0, 1] (relative
  // error 2e-7), so that the special-function unit is left to the softmax; otherwise tanh(x) = 1 - 2 / (1 + e^2x).
  template <int N>
  __device__ __forceinline__ void scores(float* s, float scale_log2) const {
    if (cap_log2 == 0.0f) {
#pragma unroll
      for (int i = 0; i < N; ++i) s[i] *= scale_log2;
      return;
    }
    float top[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < N; ++i) top[i & 3] = fmaxf(top[i & 3], fabsf(s[i]));
    const float most = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * fabsf(cap_arg);
    if (__all_sync(0xffffffffu, most <= 1.0f)) {
      constexpr float kP[7] = {0.99999994f, -0.3333284f, 0.13325198f, -0.05345685f, 0.020289687f, -0.006203149f, 0.0010409532f};
      const uint64_t arg = pack2(cap_arg, cap_arg), cap = pack2(cap_log2, cap_log2);
#pragma unroll
      for (int i = 0; i < N; i += 2) {
        const uint64_t x = mul2(pack2(s[i], s[i + 1]), arg), y = mul2(x, x);
        uint64_t p = pack2(kP[6], kP[6]);
#pragma unroll
        for (int j = 5; j >= 0; --j) p = fma2(p, y, pack2(kP[j], kP[j]));
        const float2 r = unpack2(mul2(mul2(x, cap), p));
        s[i] = r.x;
        s[i + 1] = r.y;
      }
    } else {
      const float twice = 2.0f * cap_arg * ptx::kLog2e;
#pragma unroll
      for (int i = 0; i < N; ++i) s[i] = fmaf(-2.0f * cap_log2, ptx::rcp(1.0f + ptx::ex2(s[i] * twice)), cap_log2);
    }
  }
  __host__ __device__ __forceinline__ bool plain() const { return window == kNoWindow && chunk == 0 && cap_log2 == 0.0f && out_scale == 1.0f && bias == nullptr && !sink; }
  static constexpr int kNoWindow = 1 << 30;
};

inline ScoreMods make_score_mods(const B2AttnMods* a, int heads, float scale) {
  const B2AttnMods none{0, 0, 0.0f, 1.0f, nullptr, 0};
  const B2AttnMods& b = a != nullptr ? *a : none;
  ScoreMods m{b.window > 0 ? b.window : ScoreMods::kNoWindow, b.chunk > 0 ? b.chunk : 0, 0.0f, 0.0f, b.out_scale, b.distance, heads, b.sink != 0};
  if (b.softcap > 0.0f) {
    m.cap_log2 = b.softcap * 1.4426950408889634f;
    m.cap_arg = scale / b.softcap;
  }
  return m;
}

}  // namespace b2
