// Shared by the kernels of recurrent layers with a matrix state per head: how a warp divides the key rows of a state among its
// lanes (in pairs, for packed f32 arithmetic), and the checked places of tiles and of decode rows.
#pragma once
#include <cstdint>
#include "b2/f32x2.cuh"
#include "b2/mixers.h"
#include "b2/short_conv.cuh"

namespace b2 {

// A lane holds C value columns and P pairs of key rows, RG lanes together all 2 P RG of them. RG row groups read 16 RG different
// bytes of a vector at once; more rows and fewer columns per lane read the same bytes more often, but leave less to be summed over
// the lanes. Pair p of row group rg is key rows pair_row(p, rg) and the next one.
template <int P, int RG = 16>
__device__ __forceinline__ int pair_row(int p, int rg) {
  if constexpr (P == 1) return 2 * rg;
  else return (p >> 1) * (4 * RG) + rg * 4 + (p & 1) * 2;
}
template <int P, int RG = 16>
__device__ __forceinline__ void load_pairs(const float* x, int rg, uint64_t (&v)[P]) {
  if constexpr (P == 1) {
    v[0] = *reinterpret_cast<const uint64_t*>(x + 2 * rg);
  } else {
#pragma unroll
    for (int i = 0; i < P / 2; ++i) {
      const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(x + i * (4 * RG) + rg * 4);
      v[2 * i] = t.x;
      v[2 * i + 1] = t.y;
    }
  }
}
// A lane's share of a state [d, e], from its first value column `col` on; zero outside.
template <int P, int C, int RG = 16>
__device__ __forceinline__ void load_state(const float* state, bool fresh, int d, int e, int col, int rg, uint64_t (&S)[P][C]) {
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int key = pair_row<P, RG>(p, rg);
#pragma unroll
    for (int c = 0; c < C; ++c) {
      float lo = 0.0f, hi = 0.0f;
      if (!fresh && col + c < e) {
        if (key < d) lo = state[static_cast<int64_t>(key) * e + c];
        if (key + 1 < d) hi = state[static_cast<int64_t>(key + 1) * e + c];
      }
      S[p][c] = pack2(lo, hi);
    }
  }
}
template <int P, int C, int RG = 16>
__device__ __forceinline__ void store_state(float* state, int d, int e, int col, int rg, const uint64_t (&S)[P][C]) {
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int key = pair_row<P, RG>(p, rg);
#pragma unroll
    for (int c = 0; c < C; ++c) {
      if (col + c >= e) continue;
      const float2 f = unpack2(S[p][c]);
      if (key < d) state[static_cast<int64_t>(key) * e + c] = f.x;
      if (key + 1 < d) state[static_cast<int64_t>(key + 1) * e + c] = f.y;
    }
  }
}

// The sequences [first, stop) cut into tiles of `len` rows: the sequence of tile number `tile`, or -1; `tile` becomes its number
// there. Whole warps, 32 sequences at a time.
__device__ __forceinline__ int find_tile(const B2SeqRows& sq, int first, int stop, int len, int& tile) {
  const int lane = threadIdx.x & 31;
  for (int s0 = first; s0 < stop; s0 += 32) {
    int tiles = 0;
    if (s0 + lane < stop) tiles = (max(0, sq.seq_rows[2 * (s0 + lane) + 1] - sq.seq_rows[2 * (s0 + lane)]) + len - 1) / len;
    int sum = tiles;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += up;
    }
    const uint32_t hit = __ballot_sync(0xffffffffu, tile < sum);
    if (hit != 0) {
      const int l = __ffs(hit) - 1;
      tile -= __shfl_sync(0xffffffffu, sum - tiles, l);
      return s0 + l;
    }
    tile -= __shfl_sync(0xffffffffu, sum, 31);
  }
  return -1;
}

// Sequence's decode row if the entry is in use and sound, else -1.
__device__ __forceinline__ int decode_row(const B2SeqRows& sq, int seq, ConvRow& cr, Status* status) {
  const int row = sq.seq_rows[2 * seq];
  if (row < 0 || row >= sq.rows || !cr.load(sq, seq, row, sq.banks, status)) return -1;
  return B2_ASSERT(status, cr.end == row + 1, kSiteKvIndex, row, cr.end) ? row : -1;
}

}  // namespace b2
