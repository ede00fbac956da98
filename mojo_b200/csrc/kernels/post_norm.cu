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

// The sum over a CTA of at most 32 warps; `part` alternates between calls, so that one barrier is enough.
__device__ __forceinline__ float cta_sum(float v, float* part) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = blockDim.x >> 5;
  v = warp_sum(v);
  if (n == 1) return v;
  if (lane == 0) part[warp] = v;
  __syncthreads();
  v = 0.0f;
  for (int w = 0; w < n; ++w) v += part[w];
  return v;
}

// One row of one group on its way: what is read ahead of the row's turn.
template <typename T, int VEC, int NJ>
struct RowLoad {
  float x[NJ][VEC];
  RawVec<T, VEC> y[NJ];
};

template <typename T, int VEC, int NJ, int MAXT>
__global__ void __launch_bounds__(512) post_norm_kernel(const B2PostNormArgs a, const B2SeqRows sq, int tile_rows, Status* status) {
  ptx::grid_dep_sync();
  __shared__ float part[2][32];
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
      row_first = max(b, row0 - (a.taps - 1));
    }
    if (!used) {      // rows of no sequence read as zero
      const int left = static_cast<int>(gridDim.x) - (static_cast<int>(blockIdx.x) - tile);
      const int from = seq >= 0 ? max(row0, 0) : tile, to = seq >= 0 ? min(row_end, a.rows) : a.rows, step = seq >= 0 ? 1 : left;
      for (int r = from; r < to; r += step) {
        if (seq < 0 && sq.row_seq[r] >= 0) continue;
        for (int c = base + threadIdx.x; c < stop; c += blockDim.x) {
          const float z[1] = {0.0f};
          store_f32<1>(static_cast<T*>(a.h) + static_cast<int64_t>(r) * W + c, z);
          store_f32<1>(a.x_out + static_cast<int64_t>(r) * W + c, z);
        }
      }
      return;
    }
  }

  const auto fetch = [&](int row, RowLoad<T, VEC, NJ>& in) {
    const T *emb = nullptr, *pos = nullptr;
    if (a.ids != nullptr) {
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
      for (int i = 0; i < VEC; ++i) in.x[j][i] = 0.0f;
      in.y[j].zero();
      if (c >= stop) continue;
      if (a.ids != nullptr) {
        if (emb != nullptr) load_f32<VEC>(emb + c, in.x[j]);
        if (pos != nullptr) in.y[j].load(pos + c);
      } else {
        load_f32<VEC>(a.x + static_cast<int64_t>(row) * W + c, in.x[j]);
        if (a.y != nullptr) in.y[j].load(static_cast<const T*>(a.y) + static_cast<int64_t>(row) * W + c);
      }
    }
  };

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

  RowLoad<T, VEC, NJ> in;
  fetch(row_first, in);
  for (int row = row_first; row < row_end; ++row) {
    float v[NJ][VEC], ss = 0.0f;
    const int32_t* slots = a.experts != nullptr ? a.expert_slot + static_cast<int64_t>(row) * a.top : nullptr;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = column(j);
      float u[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) u[i] = in.y[j].get(i);
      if (slots != nullptr && c < stop) {
        for (int k0 = 0; k0 < a.top; k0 += 4) {      // the rows of up to four experts are requested before the first is used
          float e[4][VEC], f[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            f[k] = 0.0f;
            if (k0 + k >= a.top) continue;
            const int slot = slots[k0 + k];
            if (!B2_ASSERT(status, slot >= 0 && slot < a.expert_rows, kSiteEpCount, slot, a.expert_rows)) {
#pragma unroll
              for (int i = 0; i < VEC; ++i) e[k][i] = 0.0f;
              continue;
            }
            f[k] = a.expert_w != nullptr ? a.expert_w[static_cast<int64_t>(row) * a.top + k0 + k] : 1.0f;
            load_f32<VEC>(static_cast<const T*>(a.experts) + static_cast<int64_t>(slot) * W + c, e[k]);
          }
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (k0 + k < a.top)
#pragma unroll
              for (int i = 0; i < VEC; ++i) u[i] = fmaf(f[k], e[k][i], u[i]);
        }
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        v[j][i] = c < stop ? fmaf(alpha, in.x[j][i], s[j][i] * u[i]) : 0.0f;
        ss = fmaf(v[j][i], v[j][i], ss);
      }
    }
    if (row + 1 < row_end) fetch(row + 1, in);
    if (a.weight != nullptr) {
      const float r = 1.0f / sqrtf(cta_sum(ss, part[row & 1]) / static_cast<float>(gw) + a.eps);
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[j][i] *= r * w[j][i];
    }
    if (a.then != nullptr) {
      float s2 = 0.0f;
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int i = 0; i < VEC; ++i) s2 = fmaf(v[j][i], v[j][i], s2);
      const float r = 1.0f / sqrtf(cta_sum(s2, part[(row & 1) ^ 1]) / static_cast<float>(gw) + a.eps);
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        float t[VEC] = {};
        if (column(j) < stop) load_f32<VEC>(a.then + column(j), t);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[j][i] *= r * t[i];
      }
    }
    const bool mine = row >= row0;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = column(j);
      float h[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        float y = cw[MAXT - 1][j][i] * v[j][i];
#pragma unroll
        for (int m = 0; m < MAXT - 1; ++m) y = fmaf(cw[m][j][i], past[m][j][i], y);
        h[i] = v[j][i] + y;
#pragma unroll
        for (int m = 0; m + 1 < MAXT - 1; ++m) past[m][j][i] = past[m + 1][j][i];
        past[MAXT - 2][j][i] = v[j][i];
      }
      if (!mine || c >= stop) continue;
      const int64_t at = a.rows_index != nullptr ? static_cast<int64_t>(blockIdx.x) : row;
      store_f32<VEC>(static_cast<T*>(a.h) + at * W + c, h);
      if (a.x_out != nullptr) store_f32<VEC>(a.x_out + static_cast<int64_t>(row) * W + c, v[j]);
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

template <typename T, int VEC, int NJ, int MAXT>
int launch(const B2PostNormArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  const int gw = a.mean_width / a.groups, vecs = (gw + VEC * NJ - 1) / (VEC * NJ), threads = (vecs + 31) / 32 * 32;
  // long tiles normalise few rows twice, short ones fill the machine
  int len = 32;
  while (len > 4 && static_cast<int64_t>(a.rows) / len * a.groups * threads < 2ll * kNumSMs * 1024) len >>= 1;
  const int tiles = a.rows_index != nullptr ? a.n_out : a.rows / len + s.seqs + 1;
  launch_pdl(post_norm_kernel<T, VEC, NJ, MAXT>, dim3(tiles, a.groups), dim3(threads), 0, stream, a, s, len, status);
  return last_launch_rc();
}
template <typename T, int VEC, int NJ>
int by_taps(const B2PostNormArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  return a.taps <= 4 || a.conv_w == nullptr ? launch<T, VEC, NJ, 4>(a, s, status, stream) : launch<T, VEC, NJ, kMaxTaps>(a, s, status, stream);
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
