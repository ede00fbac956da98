// What an attention layer does beyond plain causal softmax: a sliding window, a soft cap on the scores, a factor on the result.
#pragma once
#include "b2/ptx.cuh"

namespace b2 {

struct ScoreMods {
  int window;         // positions a row sees, its own included
  float cap_log2;     // cap * log2(e); 0: no cap
  float cap_arg;      // 2 log2(e) * scale / cap: twice the argument of tanh, in powers of two
  float out_scale;

  // log2(e) * score of a raw dot product: capped as cap * tanh(x) = cap - 2 cap / (1 + e^2x), or scaled
  __device__ __forceinline__ float score(float dot, float scale_log2) const {
    if (cap_log2 == 0.0f) return dot * scale_log2;
    return fmaf(-2.0f * cap_log2, ptx::rcp(1.0f + ptx::ex2(dot * cap_arg)), cap_log2);
  }
  __host__ __device__ __forceinline__ bool plain() const { return window == kNoWindow && cap_log2 == 0.0f && out_scale == 1.0f; }
  static constexpr int kNoWindow = 1 << 30;
};

// window <= 0: everything; softcap <= 0: none.
inline ScoreMods make_score_mods(int window, float softcap, float out_scale, float scale) {
  const float log2e = 1.4426950408889634f;
  ScoreMods m{window > 0 ? window : ScoreMods::kNoWindow, 0.0f, 0.0f, out_scale};
  if (softcap > 0.0f) {
    m.cap_log2 = softcap * log2e;
    m.cap_arg = 2.0f * log2e * scale / softcap;
  }
  return m;
}

}  // namespace b2
