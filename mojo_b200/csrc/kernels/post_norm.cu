// A residual that is normalised after the sum, with a short convolution over time on what a sublayer reads. One kernel between
// any two sublayers: x <- norm(alpha x + scale (what the finished one produced)), h = x + conv(x). The norm treats runs of columns
// (groups) one by one and the convolution channels, so a CTA takes one group of a tile of consecutive rows of one sequence. It
// walks over the rows, a thread on the same columns all the way with the convolution's past in registers; the few rows ahead of
// the tile are normalised again instead of being passed between CTAs, which is why the new stream goes to another buffer than the
// old one.
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/recurrence.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kMaxTop = 32;
constexpr int kMaxTaps = 16;

// R sums over a CTA of at most 32 warps; `part` alternates between calls, so that one barrier is enough.
template <int R>
__device__ __forceinline__ void cta_sums(float (&v)[R], float (*part)[32]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = blockDim.x >> 5;
  if constexpr (R == 4) {
    warp_sum4(v);
  } else {
#pragma unroll
    for (int r = 0; r < R; ++r) v[r] = warp_sum(v[r]);
  }
  if (n == 1) return;
  if (lane == 0) {
#pragma unroll
    for (int r = 0; r < R; ++r) part[r][warp] = v[r];
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < R; ++r) v[r] = 0.0f;
  for (int w = 0; w < n; ++w)
#pragma unroll
    for (int r = 0; r < R; ++r) v[r] += part[r][w];
}

template <typename T, int VEC, int NJ, int MAXT, int RB>
__global__ void __launch_bounds__(512) post_norm_kernel(const B2PostNormArgs a, const B2SeqRows sq, int tile_rows, Status* status) {
  ptx::grid_dep_sync();
  __shared__ float part[2][RB][32];
  extern __shared__ int32_t choice_sm[];      // expert rows of the tile [rows][top], then their weights
  const int gw = a.mean_width / a.groups, base = blockIdx.y * gw, stop = base + gw, W = a.width;
  const auto column = [&](int j) { return base + static_cast<int>(threadIdx.x + j * blockDim.x) * VEC; };

  // the rows of this CTA: [row0, row_end) are written, those from row_first on are normalised
  int row0, row_end, row_first;
  ConvRow cr{};
  if (a.rows_index != nullptr) {
    const int64_t row = a.rows_index[blockIdx.x];
    if (!B2_ASSERT(status, row >= 0 && row < a.rows, kSiteKvIndex, row, a.rows)) return;
    row0 = row_first = static_cast<int>(row);
    row_end = row0 + 1;
  } else {
    int tile = static_cast<int>(blockIdx.x);
    const int seq = find_tile(sq, 0, sq.seqs, tile_rows, tile);
    bool used = false;
    if (seq >= 0) {
      const int b = sq.seq_rows[2 * seq], e = sq.seq_rows[2 * seq + 1];
      row0 = b + tile * tile_rows;
      row_end = min(row0 + tile_rows, e);
      used = cr.load(sq, seq, row0, sq.banks, status);
      row_first = a.conv_w != nullptr ? max(b, row0 - (a.taps - 1)) : row0;
    }
    if (!used) {      // rows of no sequence read as zero
      // an unused sequence's tile, or one of the CTAs past the last tile, which look for such rows 32 at a time
      const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
      const int spare = static_cast<int>(gridDim.x) - (static_cast<int>(blockIdx.x) - tile);
      const int from = seq >= 0 ? max(row0, 0) + warp * 32 : (tile * n_warps + warp) * 32, to = seq >= 0 ? min(row_end, a.rows) : a.rows;
      for (int r0 = from; r0 < to; r0 += (seq >= 0 ? 1 : spare) * n_warps * 32) {
        const bool empty = r0 + lane < to && (seq >= 0 || sq.row_seq[r0 + lane] < 0);
        for (uint32_t rows = __ballot_sync(0xffffffffu, empty); rows != 0; rows &= rows - 1) {
          const int64_t at = static_cast<int64_t>(r0 + __ffs(rows) - 1) * W;
          for (int c = base + lane; c < stop; c += 32) {
            const float z[1] = {0.0f};
            store_f32<1>(static_cast<T*>(a.h) + at + c, z);
            store_f32<1>(a.x_out + at + c, z);
          }
        }
      }
      return;
    }
  }

  const bool starts = a.ids != nullptr;
  const float alpha = starts ? 1.0f : a.alpha;
  float w[NJ][VEC], s[NJ][VEC], cw[MAXT][NJ][VEC], past[MAXT - 1][NJ][VEC];
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = column(j);
    const bool in = c < stop;
#pragma unroll
    for (int i = 0; i < VEC; ++i) w[j][i] = s[j][i] = 1.0f;
    if (in && a.weight != nullptr) load_f32<VEC>(a.weight + c, w[j]);
    if (in && a.y_scale != nullptr && !starts) load_f32<VEC>(a.y_scale + c, s[j]);
    // taps and past are those of MAXT taps, the oldest ones zero
#pragma unroll
    for (int m = 0; m < MAXT; ++m) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) cw[m][j][i] = 0.0f;
      const int tap = m - (MAXT - a.taps);
      if (in && a.conv_w != nullptr && tap >= 0) load_f32<VEC>(a.conv_w + static_cast<int64_t>(tap) * W + c, cw[m][j]);
    }
#pragma unroll
    for (int m = 0; m < MAXT - 1; ++m) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) past[m][j][i] = 0.0f;
      const int back = MAXT - 1 - m;      // rows ahead of row_first
      if (in && a.conv_w != nullptr && row_first == cr.begin && cr.rd >= 0 && back <= a.taps - 1)
        load_f32<VEC>(a.conv_state + (static_cast<int64_t>(cr.rd) * (a.taps - 1) + a.taps - 1 - back) * W + c, past[m][j]);
    }
  }

  float* choice_w = reinterpret_cast<float*>(choice_sm + (tile_rows + a.taps) * a.top);
  if (a.experts != nullptr) {
    const int64_t from = static_cast<int64_t>(row_first) * a.top;
    for (int i = threadIdx.x; i < (row_end - row_first) * a.top; i += blockDim.x) {
      const int slot = a.expert_slot[from + i];
      const bool ok = B2_ASSERT(status, slot >= 0 && slot < a.expert_rows, kSiteEpCount, slot, a.expert_rows);
      choice_sm[i] = ok ? slot : 0;
      choice_w[i] = !ok ? 0.0f : a.expert_w != nullptr ? a.expert_w[from + i] : 1.0f;
    }
    __syncthreads();
  }

  int turn = 0;
  for (int first = row_first; first < row_end; first += RB, turn ^= 1) {
    // RB rows at a time: all their loads are in flight together, and their sums share a barrier
    float v[RB][NJ][VEC], ss[RB];
    RawVec<T, VEC> y[RB][NJ];
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      const int row = first + r;
      const T *emb = nullptr, *pos = nullptr;
      if (starts && row < row_end) {
        const int64_t id = a.ids[row];
        if (B2_ASSERT(status, id >= 0 && id < a.vocab, kSiteKvIndex, id, a.vocab)) emb = static_cast<const T*>(a.embed) + id * W;
        if (a.pos_table != nullptr) {
          const int p = a.positions[row];
          if (B2_ASSERT(status, p >= 0 && p < a.max_pos, kSiteKvIndex, p, a.max_pos)) pos = static_cast<const T*>(a.pos_table) + static_cast<int64_t>(p) * W;
        }
      }
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int c = column(j);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[r][j][i] = 0.0f;
        y[r][j].zero();
        if (c >= stop || row >= row_end) continue;
        if (starts) {
          if (emb != nullptr) load_f32<VEC>(emb + c, v[r][j]);
          if (pos != nullptr) y[r][j].load(pos + c);
        } else {
          load_f32<VEC>(a.x + static_cast<int64_t>(row) * W + c, v[r][j]);
          if (a.y != nullptr) y[r][j].load(static_cast<const T*>(a.y) + static_cast<int64_t>(row) * W + c);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = column(j);
      float u[RB][VEC];
#pragma unroll
      for (int r = 0; r < RB; ++r)
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[r][i] = y[r][j].get(i);
      if (a.experts != nullptr && c < stop) {
        constexpr int kAhead = RB >= 4 ? 2 : 4;      // experts of a row on their way at a time
        const T* rows = static_cast<const T*>(a.experts) + c;
        for (int k0 = 0; k0 < a.top; k0 += kAhead) {
          RawVec<T, VEC> e[RB][kAhead];
#pragma unroll
          for (int r = 0; r < RB; ++r)
#pragma unroll
            for (int k = 0; k < kAhead; ++k) {
              e[r][k].zero();
              if (first + r < row_end && k0 + k < a.top) e[r][k].load(rows + static_cast<int64_t>(choice_sm[(first + r - row_first) * a.top + k0 + k]) * W);
            }
#pragma unroll
          for (int r = 0; r < RB; ++r)
#pragma unroll
            for (int k = 0; k < kAhead; ++k) {
              if (first + r >= row_end || k0 + k >= a.top) continue;
              const float f = choice_w[(first + r - row_first) * a.top + k0 + k];
#pragma unroll
              for (int i = 0; i < VEC; ++i) u[r][i] = fmaf(f, e[r][k].get(i), u[r][i]);
            }
        }
      }
#pragma unroll
      for (int r = 0; r < RB; ++r)
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[r][j][i] = c < stop ? fmaf(alpha, v[r][j][i], s[j][i] * u[r][i]) : 0.0f;
    }
    const auto normalise = [&](auto weight_of, int t) {
#pragma unroll
      for (int r = 0; r < RB; ++r) {
        ss[r] = 0.0f;
#pragma unroll
        for (int j = 0; j < NJ; ++j)
#pragma unroll
          for (int i = 0; i < VEC; ++i) ss[r] = fmaf(v[r][j][i], v[r][j][i], ss[r]);
      }
      cta_sums<RB>(ss, part[t]);
#pragma unroll
      for (int r = 0; r < RB; ++r) {
        const float f = 1.0f / sqrtf(ss[r] / static_cast<float>(gw) + a.eps);
#pragma unroll
        for (int j = 0; j < NJ; ++j)
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[r][j][i] *= f * weight_of(j, i);
      }
    };
    if (a.weight != nullptr) normalise([&](int j, int i) { return w[j][i]; }, turn);
    if (a.then != nullptr) {      // one row per CTA then
#pragma unroll
      for (int j = 0; j < NJ; ++j)
        if (column(j) < stop) load_f32<VEC>(a.then + column(j), w[j]);
      normalise([&](int j, int i) { return w[j][i]; }, turn ^ 1);
    }
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      const int row = first + r;
      if (row >= row_end) break;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int c = column(j);
        float h[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          float y = cw[MAXT - 1][j][i] * v[r][j][i];
#pragma unroll
          for (int m = 0; m < MAXT - 1; ++m) y = fmaf(cw[m][j][i], past[m][j][i], y);
          h[i] = v[r][j][i] + y;
#pragma unroll
          for (int m = 0; m + 1 < MAXT - 1; ++m) past[m][j][i] = past[m + 1][j][i];
          past[MAXT - 2][j][i] = v[r][j][i];
        }
        if (row < row0 || c >= stop) continue;
        const int64_t at = a.rows_index != nullptr ? static_cast<int64_t>(blockIdx.x) : row;
        store_f32<VEC>(static_cast<T*>(a.h) + at * W + c, h);
        if (a.x_out != nullptr) store_f32<VEC>(a.x_out + static_cast<int64_t>(row) * W + c, v[r][j]);
      }
    }
  }
  // the tile with a sequence's last row leaves what the next step's convolution will read
  if (a.conv_w != nullptr && a.taps > 1 && row_end == cr.end) {
#pragma unroll
    for (int m = 0; m < MAXT - 1; ++m) {
      const int at = m - (MAXT - a.taps);
      if (at < 0) continue;
#pragma unroll
      for (int j = 0; j < NJ; ++j)
        if (column(j) < stop) store_f32<VEC>(a.conv_state + (static_cast<int64_t>(cr.wr) * (a.taps - 1) + at) * W + column(j), past[m][j]);
    }
  }
}

template <typename T, int VEC, int NJ, int MAXT, int RB>
int launch(const B2PostNormArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  const int gw = a.mean_width / a.groups, vecs = (gw + VEC * NJ - 1) / (VEC * NJ), threads = (vecs + 31) / 32 * 32;
  // long tiles normalise few rows twice, short ones fill the machine; with the rows ahead a tile is a multiple of RB rows
  int len = a.rows <= s.seqs || a.rows_index != nullptr ? 1 : 16;
  if (RB > 1) {
    const int ahead = a.conv_w != nullptr ? a.taps - 1 : 0;
    for (int most = 32; most >= 4; most -= most > 16 ? 16 : 4) {
      len = most - ahead % RB;
      if (static_cast<int64_t>(a.rows) / len * a.groups * threads >= 8ll * kNumSMs * 128) break;
    }
  }
  const int tiles = a.rows_index != nullptr ? a.n_out : a.rows / len + s.seqs + 1;
  const int smem = a.experts != nullptr ? (len + a.taps) * a.top * 8 : 0;
  launch_pdl(post_norm_kernel<T, VEC, NJ, MAXT, RB>, dim3(tiles, a.groups), dim3(threads), smem, stream, a, s, len, status);
  return last_launch_rc();
}
template <typename T, int VEC, int NJ>
int by_taps(const B2PostNormArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  if (a.taps > 4 && a.conv_w != nullptr) return launch<T, VEC, NJ, kMaxTaps, 1>(a, s, status, stream);
  if constexpr (NJ > 2) return launch<T, VEC, NJ, 4, 1>(a, s, status, stream);
  else return a.rows_index != nullptr || a.rows <= s.seqs ? launch<T, VEC, NJ, 4, 1>(a, s, status, stream) : launch<T, VEC, NJ, 4, 4 / NJ>(a, s, status, stream);
}
template <typename T>
int dispatch(const B2PostNormArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  const int gw = a.mean_width / a.groups;
  if (gw % 4 == 0 && a.width % 4 == 0) {
    if (gw <= 4 * 512) return by_taps<T, 4, 1>(a, s, status, stream);
    if (gw <= 8 * 512) return by_taps<T, 4, 2>(a, s, status, stream);
    return gw <= 16 * 512 ? by_taps<T, 4, 4>(a, s, status, stream) : -kTooLarge;
  }
  if (gw <= 512) return by_taps<T, 1, 1>(a, s, status, stream);
  return gw <= 8 * 512 ? by_taps<T, 1, 8>(a, s, status, stream) : -kTooLarge;
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_post_norm(const B2PostNormArgs* a, const B2SeqRows* s, int f32, Status* status, cudaStream_t stream) {
  if (a->rows <= 0 || a->n_out <= 0) return 0;
  if (a->width <= 0 || a->mean_width <= 0 || a->mean_width > a->width || a->groups < 1 || a->groups > 65535 || a->mean_width % a->groups != 0 || a->h == nullptr ||
      (a->ids == nullptr && a->x == nullptr) || (a->ids != nullptr && a->embed == nullptr) || (a->pos_table != nullptr && (a->ids == nullptr || a->positions == nullptr)) ||
      (a->experts != nullptr && (a->expert_slot == nullptr || a->top < 1 || a->top > kMaxTop)) || (a->x_out != nullptr && a->x_out == a->x) ||
      (a->rows_index != nullptr ? a->conv_w != nullptr || a->x_out != nullptr : s->rows != a->rows || a->x_out == nullptr || a->n_out != a->rows) ||
      (a->conv_w != nullptr && (a->taps < 1 || a->taps > kMaxTaps || (a->taps > 1 && a->conv_state == nullptr))))
    return -kBadArgument;
  return f32 ? dispatch<float>(*a, *s, status, stream) : dispatch<__nv_bfloat16>(*a, *s, status, stream);
}
