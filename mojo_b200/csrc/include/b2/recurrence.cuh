// Shared by the kernels of recurrent layers with a matrix state per head: packed f32 arithmetic on pairs of key rows, how a
// half-warp divides the key rows of a state among its lanes, and the checked place of a decode row.
#pragma once
#include <cstdint>
#include "b2/mixers.h"
#include "b2/short_conv.cuh"

namespace b2 {

// Packed pairs of f32 (two key rows): one instruction per two multiply-adds.
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ float half_sum(uint64_t v) {
  const float2 f = unpack2(v);
  return f.x + f.y;
}

// A lane holds four value columns and P pairs of key rows (32 P rows in all). The 16 row groups of a half-warp read 256 different
// bytes of a vector at once; a mapping with more rows and fewer columns per lane reads the same bytes more often, and
// shared-memory bandwidth is what two CTAs on one SM run short of first.
// Pair p of row group rg is key rows pair_row(p, rg) and the next one.
template <int P>
__device__ __forceinline__ int pair_row(int p, int rg) {
  if constexpr (P == 1) return 2 * rg;
  else return (p >> 1) * 64 + rg * 4 + (p & 1) * 2;
}
template <int P>
__device__ __forceinline__ void load_pairs(const float* x, int rg, uint64_t (&v)[P]) {
  if constexpr (P == 1) {
    v[0] = *reinterpret_cast<const uint64_t*>(x + 2 * rg);
  } else {
#pragma unroll
    for (int i = 0; i < P / 2; ++i) {
      const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(x + i * 64 + rg * 4);
      v[2 * i] = t.x;
      v[2 * i + 1] = t.y;
    }
  }
}
// A lane's share of a state [d, e], from its first value column `col` on; zero outside.
template <int P>
__device__ __forceinline__ void load_state(const float* state, bool fresh, int d, int e, int col, int rg, uint64_t (&S)[P][4]) {
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int key = pair_row<P>(p, rg);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      float lo = 0.0f, hi = 0.0f;
      if (!fresh && col + c < e) {
        if (key < d) lo = state[static_cast<int64_t>(key) * e + c];
        if (key + 1 < d) hi = state[static_cast<int64_t>(key + 1) * e + c];
      }
      S[p][c] = pack2(lo, hi);
    }
  }
}
template <int P>
__device__ __forceinline__ void store_state(float* state, int d, int e, int col, int rg, const uint64_t (&S)[P][4]) {
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int key = pair_row<P>(p, rg);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      if (col + c >= e) continue;
      const float2 f = unpack2(S[p][c]);
      if (key < d) state[static_cast<int64_t>(key) * e + c] = f.x;
      if (key + 1 < d) state[static_cast<int64_t>(key + 1) * e + c] = f.y;
    }
  }
}

// Sequence's decode row if the entry is in use and sound, else -1.
__device__ __forceinline__ int decode_row(const B2SeqRows& sq, int seq, ConvRow& cr, Status* status) {
  const int row = sq.seq_rows[2 * seq];
  if (row < 0 || row >= sq.rows || !cr.load(sq, seq, row, sq.banks, status)) return -1;
  return B2_ASSERT(status, cr.end == row + 1, kSiteKvIndex, row, cr.end) ? row : -1;
}

}  // namespace b2
