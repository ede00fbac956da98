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

// VEC raw elements in registers.
template <typename T, int VEC>
struct RawVec {
  float v[VEC];
  __device__ __forceinline__ void load(const T* p) { load_f32<VEC>(p, v); }
  __device__ __forceinline__ void store(T* p) const { store_f32<VEC>(p, v); }
  __device__ __forceinline__ void zero() {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = 0.0f;
  }
  __device__ __forceinline__ void set(T a, T b) { v[0] = a; v[1] = b; }
  __device__ __forceinline__ float get(int i) const { return v[i]; }
};
template <>
struct RawVec<__nv_bfloat16, 4> {
  uint2 v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint2*>(p); }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *reinterpret_cast<uint2*>(p) = v; }
  __device__ __forceinline__ void zero() { v = make_uint2(0, 0); }
  __device__ __forceinline__ float get(int i) const {
    const uint32_t w = i < 2 ? v.x : v.y;
    return i & 1 ? ptx::bf16_hi(w) : ptx::bf16_lo(w);
  }
};

template <>
struct RawVec<__nv_bfloat16, 2> {
  uint32_t v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint32_t*>(p); }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *reinterpret_cast<uint32_t*>(p) = v; }
  __device__ __forceinline__ void zero() { v = 0; }
  __device__ __forceinline__ void set(__nv_bfloat16 a, __nv_bfloat16 b) {
    v = static_cast<uint32_t>(__bfloat16_as_ushort(a)) | static_cast<uint32_t>(__bfloat16_as_ushort(b)) << 16;
  }
  __device__ __forceinline__ float get(int i) const { return i & 1 ? ptx::bf16_hi(v) : ptx::bf16_lo(v); }
};

// The convolution of `n` (<= TT) consecutive rows of one sequence for VEC channels: the whole window is fetched at once, so
// that its loads are in flight together, and every row is fetched once. `save` also writes the next step's bank.
// TAPS == 0: any number of taps, row by row.
template <typename T, int VEC, int TAPS, int TT>
__device__ __forceinline__ void conv_rows(const ConvSource<T>& s, const ConvRow& r, int row0, int n, int chan, bool save, float (&y)[TT][VEC]) {
  if constexpr (TAPS == 0) {
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      if (t < n) {
        s.template apply<VEC>(r, row0 + t, chan, y[t]);
        if (save) s.template save<VEC>(r, row0 + t, chan);
      } else {
#pragma unroll
        for (int v = 0; v < VEC; ++v) y[t][v] = 0.0f;
      }
    }
  } else {
    RawVec<T, VEC> u[TT + TAPS - 1];
    // inside a sequence, away from its first and last rows of the step, nothing but projection rows is touched
    const bool interior = n == TT && row0 - (TAPS - 1) >= r.begin && r.end - row0 >= TT + TAPS - 1;
    if (interior) {
      const T* p = s.proj + static_cast<int64_t>(row0 - (TAPS - 1)) * s.ld + chan;
#pragma unroll
      for (int i = 0; i < TT + TAPS - 1; ++i, p += s.ld) u[i].load(p);
    } else {
#pragma unroll
      for (int i = 0; i < TT + TAPS - 1; ++i) {
        const int src = row0 - (TAPS - 1) + i;
        const T* p = src >= r.begin ? s.proj + src * s.ld + chan : r.rd >= 0 ? s.bank(r.rd, TAPS - 1 - (r.begin - src), chan) : nullptr;
        if (i < n + TAPS - 1 && p != nullptr) u[i].load(p);
        else u[i].zero();
      }
    }
    float w[TAPS][VEC];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_f32<VEC>(s.w + static_cast<int64_t>(j) * s.channels + chan, w[j]);
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        float a = 0.0f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) a = fmaf(w[j][v], u[t + j].get(v), a);
        y[t][v] = a;
      }
    if (save && !interior) {
#pragma unroll
      for (int t = 0; t < TT; ++t)
        if (t < n && r.end - (row0 + t) <= TAPS - 1) u[t + TAPS - 1].store(s.bank(r.wr, TAPS - 1 - (r.end - (row0 + t)), chan));
      const int total = r.end - r.begin;
      if (row0 == r.begin && total < TAPS - 1) {       // older part of the history moves over
#pragma unroll
        for (int i = 0; i < TAPS - 1; ++i)
          if (i >= total) u[i].store(s.bank(r.wr, i - total, chan));
      }
    }
  }
}

}  // namespace b2
