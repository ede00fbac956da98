// Short causal convolution over time, per channel, for kernels that apply it while they read a projection:
// y[t] = sum_j w[j] u[t - taps + 1 + j], where u comes from this step's rows or, before the sequence's first row of the
// step, from its state bank (the last taps - 1 projected values, oldest first), or is zero before the sequence's start.
#pragma once
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/mixers.h"

namespace b2 {

// One row's place in its sequence: the sequence's rows of this step and the banks it reads and writes.
struct ConvRow {
  int begin, end, rd, wr;
  __device__ __forceinline__ bool load(const B2SeqRows& s, int seq, int row, int banks, Status* status) {
    begin = s.seq_rows[2 * seq];
    end = s.seq_rows[2 * seq + 1];
    rd = s.seq_state[2 * seq];
    wr = s.seq_state[2 * seq + 1];
    if (wr < 0) return false;      // unused entry
    return B2_ASSERT(status, wr < banks && rd < banks && begin >= 0 && row >= begin && row < end && end <= s.rows, kSiteKvIndex, row, wr);
  }
};

template <typename T>
struct ConvSource {
  const T* proj;
  int64_t ld;
  const float* w;      // [taps, channels]
  T* state;            // [banks, taps - 1, channels]
  int taps, channels, banks;

  __device__ __forceinline__ T* bank(int b, int m, int chan) const {
    return state + (static_cast<int64_t>(b) * (taps - 1) + m) * channels + chan;
  }
  template <int VEC>
  __device__ __forceinline__ void apply(const ConvRow& r, int row, int chan, float (&y)[VEC]) const {
#pragma unroll
    for (int v = 0; v < VEC; ++v) y[v] = 0.0f;
    for (int j = 0; j < taps; ++j) {
      const int src = row - taps + 1 + j;
      float u[VEC], k[VEC];
      if (src >= r.begin) {
        load_f32<VEC>(proj + src * ld + chan, u);
      } else if (r.rd >= 0) {
        load_f32<VEC>(bank(r.rd, taps - 1 - (r.begin - src), chan), u);
      } else {
        continue;
      }
      load_f32<VEC>(w + static_cast<int64_t>(j) * channels + chan, k);
#pragma unroll
      for (int v = 0; v < VEC; ++v) y[v] = fmaf(k[v], u[v], y[v]);
    }
  }
  // This row's share of the bank the next step will read. Every (row, channel) is saved by exactly one thread, or by
  // several that write the same value.
  template <int VEC>
  __device__ __forceinline__ void save(const ConvRow& r, int row, int chan) const {
    const int keep = taps - 1;
    if (r.end - row <= keep) {
      float u[VEC];
      load_f32<VEC>(proj + row * ld + chan, u);
      store_f32<VEC>(bank(r.wr, keep - (r.end - row), chan), u);
    }
    const int n = r.end - r.begin;
    if (row == r.begin && n < keep) {        // a step shorter than the history: its older part moves over
      for (int m = 0; m < keep - n; ++m) {
        float u[VEC] = {};
        if (r.rd >= 0) load_f32<VEC>(bank(r.rd, m + n, chan), u);
        store_f32<VEC>(bank(r.wr, m, chan), u);
      }
    }
  }
};

}  // namespace b2
