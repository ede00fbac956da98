// What an attention layer does beyond plain causal softmax: a sliding window, a soft cap on the scores, a factor on the result.
#pragma once
#include "b2/f32x2.cuh"
#include "b2/ptx.cuh"

namespace b2 {

struct ScoreMods {
  int window;         // positions a row sees, its own included
  float cap_log2;     // cap * log2(e); 0: no cap
  float cap_arg;      // scale / cap
  float out_scale;

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
  __host__ __device__ __forceinline__ bool plain() const { return window == kNoWindow && cap_log2 == 0.0f && out_scale == 1.0f; }
  static constexpr int kNoWindow = 1 << 30;
};

// window <= 0: everything; softcap <= 0: none.
inline ScoreMods make_score_mods(int window, float softcap, float out_scale, float scale) {
  ScoreMods m{window > 0 ? window : ScoreMods::kNoWindow, 0.0f, 0.0f, out_scale};
  if (softcap > 0.0f) {
    m.cap_log2 = softcap * 1.4426950408889634f;
    m.cap_arg = scale / softcap;
  }
  return m;
}

}  // namespace b2
