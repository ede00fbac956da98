// Front ends with short causal convolutions over time. For attention: causal convolution over time on every q, k and v channel, rotary
// embedding, RMS norm of the q and k heads, scatter of k and v into the paged cache. One warp owns one head and a few
// consecutive rows. What the convolution needs from before the step comes from the sequence's state bank; the step's last
// taps - 1 projected rows go to its other bank, so no warp reads what another one of the same launch writes.
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/recurrence.cuh"
#include "b2/short_conv.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kMaxHead = 256;
constexpr int kWarps = 8;

// A warp's rows: runs of rows of one sequence, each convolved at once (`conv_rows`), then rotated and normalised row by row.
template <typename T, int VEC, int NJ, int TAPS, int TT>
__global__ void __launch_bounds__(kWarps * 32, TAPS > 0 && NJ == 1 ? 3 : 1) conv_qkv_kernel(const B2ConvQkvArgs a, const B2SeqRows sq, Status* status) {
  ptx::grid_dep_sync();
  __shared__ __align__(16) float head_sm[kWarps][kMaxHead];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * kWarps + warp;
  const int n_heads = a.heads + 2 * a.kv_heads;
  if (head >= n_heads) return;
  const bool is_q = head < a.heads, is_v = head >= a.heads + a.kv_heads;
  const int kvh = is_q ? 0 : head - a.heads - (is_v ? a.kv_heads : 0);
  const int dim = is_v ? a.vdim : a.dim, pad = is_v ? a.pad_vdim : a.pad_dim;
  const int chan0 = is_q ? head * a.dim : is_v ? (a.heads + a.kv_heads) * a.dim + kvh * a.vdim : (a.heads + kvh) * a.dim;
  const int channels = (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim;
  const int half = a.rot >> 1;
  const ConvSource<T> src{static_cast<const T*>(a.proj), a.ld, a.conv_w, static_cast<T*>(a.conv_state), a.taps, channels, sq.banks};
  float* hs = head_sm[warp];
  const float inv_dim = 1.0f / static_cast<float>(dim);
  const int row_end = min(sq.rows, static_cast<int>(blockIdx.x + 1) * TT);
  int run = 0;
  for (int row0 = blockIdx.x * TT; row0 < row_end; row0 += run) {
    run = 1;
    const int seq = sq.row_seq[row0];
    ConvRow cr;
    const bool valid = seq >= 0 && B2_ASSERT(status, seq < sq.seqs, kSiteKvIndex, seq, sq.seqs) && cr.load(sq, seq, row0, sq.banks, status);
    if (!valid) {      // padding row
      if (is_q)
        for (int e = lane; e < pad; e += 32) {
          const float z[1] = {0.0f};
          store_f32<1>(static_cast<T*>(a.q_out) + (static_cast<int64_t>(row0) * a.heads + head) * a.pad_dim + e, z);
        }
      continue;
    }
    run = min(row_end, cr.end) - row0;
    float val[NJ][TT][VEC];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int e = (lane + 32 * j) * VEC;
      if (e < dim) {
        conv_rows<T, VEC, TAPS, TT>(src, cr, row0, run, chan0 + e, true, val[j]);
      } else {
#pragma unroll
        for (int t = 0; t < TT; ++t)
#pragma unroll
          for (int v = 0; v < VEC; ++v) val[j][t][v] = 0.0f;
      }
    }
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      if (t >= run) break;
      const int row = row0 + t;
      if (!is_v) {
        // rotate pairs (i, i + rot / 2), then divide by the root mean square of the head
        int pos = a.positions[row];
        if (!B2_ASSERT(status, pos >= 0 && pos < a.max_pos, kSiteKvIndex, pos, a.max_pos)) pos = 0;
        const float* cs = a.cos_sin + static_cast<int64_t>(pos) * a.rot;
        __syncwarp();
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const int e = (lane + 32 * j) * VEC;
          if (e < dim) store_f32<VEC>(hs + e, val[j][t]);
        }
        __syncwarp();
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const int e0 = (lane + 32 * j) * VEC;
          if (half % VEC == 0) {      // a vector lies on one side of the rotated span
            if (e0 < a.rot) {
              const bool lo = e0 < half;
              float c[VEC], sn[VEC], other[VEC];
              load_f32<VEC>(cs + (lo ? e0 : e0 - half), c);
              load_f32<VEC>(cs + (lo ? half + e0 : e0), sn);
              load_f32<VEC>(hs + (lo ? e0 + half : e0 - half), other);
#pragma unroll
              for (int v = 0; v < VEC; ++v) val[j][t][v] = val[j][t][v] * c[v] + (lo ? -other[v] : other[v]) * sn[v];
            }
          } else {
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
              const int e = e0 + v;
              if (e < half) val[j][t][v] = val[j][t][v] * cs[e] - hs[e + half] * cs[half + e];
              else if (e < a.rot) val[j][t][v] = val[j][t][v] * cs[e - half] + hs[e - half] * cs[e];
            }
          }
#pragma unroll
          for (int v = 0; v < VEC; ++v) ss = fmaf(val[j][t][v], val[j][t][v], ss);      // 0 past dim
        }
        ss = warp_sum(ss);
        const float r = rsqrtf(ss * inv_dim + a.eps);
#pragma unroll
        for (int j = 0; j < NJ; ++j)
#pragma unroll
          for (int v = 0; v < VEC; ++v) val[j][t][v] *= r;
      }
      T* dst;
      int lim = pad;          // queries: zeros up to the padded size; cache rows are zero there from the start
      if (is_q) {
        dst = static_cast<T*>(a.q_out) + (static_cast<int64_t>(row) * a.heads + head) * a.pad_dim;
      } else {
        const int64_t slot = a.slots[row];
        if (slot < 0 || !B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots)) continue;
        T* cache = static_cast<T*>(is_v ? a.v_cache : a.k_cache);
        const uint32_t page = static_cast<uint32_t>(slot) / static_cast<uint32_t>(a.page_size);      // the host keeps slots below 2^31
        const uint32_t in_page = static_cast<uint32_t>(slot) - page * a.page_size;
        dst = cache + ((static_cast<int64_t>(page) * a.kv_heads + kvh) * a.page_size + in_page) * pad;
        lim = dim;
      }
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int e = (lane + 32 * j) * VEC;
        if (e < lim) store_f32<VEC>(dst + e, val[j][t]);
      }
      if (is_q)
        for (int e = 32 * NJ * VEC + lane; e < pad; e += 32) { const float z[1] = {0.0f}; store_f32<1>(dst + e, z); }
    }
  }
}

// The common case (4 taps, head sizes up to 128 and multiples of 4). Work unit = (tile of TT rows, head); every warp takes
// the same number of consecutive units, heads first, so that it keeps a tile's rotary factors in registers across heads.
// Rotation partners come from another lane. Tiles that cross a sequence border go row by row.
struct RowLane {
  int lane, e0, half, partner;
  bool turns, lo;
};
template <int TT>
struct RowFactors {
  float cs[TT][4], sn[TT][4];
  int cell[TT];      // cache row of head 0 (heads of a page lie page_size apart); -1: nothing is cached
  __device__ __forceinline__ void load(const B2ConvQkvArgs& a, const RowLane& l, int row0, int n, bool valid, Status* status) {
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      cell[t] = -1;
#pragma unroll
      for (int v = 0; v < 4; ++v) {
        cs[t][v] = 1.0f;
        sn[t][v] = 0.0f;
      }
      if (!valid || t >= n) continue;
      if (l.turns) {
        int pos = a.positions[row0 + t];
        if (!B2_ASSERT(status, pos >= 0 && pos < a.max_pos, kSiteKvIndex, pos, a.max_pos)) pos = 0;
        const float* p = a.cos_sin + static_cast<int64_t>(pos) * a.rot + (l.lo ? l.e0 : l.e0 - l.half);
        load_f32<4>(p, cs[t]);
        load_f32<4>(p + l.half, sn[t]);
        if (l.lo) {
#pragma unroll
          for (int v = 0; v < 4; ++v) sn[t][v] = -sn[t][v];
        }
      }
      if (a.kv_heads > 0) {
        const int64_t slot = a.slots[row0 + t];
        if (slot >= 0 && B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots)) {
          // the host keeps num_slots * kv_heads below 2^31
          const uint32_t page = static_cast<uint32_t>(slot) / static_cast<uint32_t>(a.page_size);
          cell[t] = static_cast<int>(page * a.kv_heads * a.page_size + (static_cast<uint32_t>(slot) - page * a.page_size));
        }
      }
    }
  }
};

// `n` rows from row0 (all of one sequence; valid == false: one padding row) of one head.
template <typename T, int TT>
__device__ __forceinline__ void conv_head(const B2ConvQkvArgs& a, const ConvSource<T>& src, const ConvRow& cr, bool valid, int row0, int n, int head,
                                          const RowLane& l, const RowFactors<TT>& f) {
  const bool is_q = head < a.heads, is_v = head >= a.heads + a.kv_heads;
  const int kvh = is_q ? 0 : head - a.heads - (is_v ? a.kv_heads : 0);
  const int dim = is_v ? a.vdim : a.dim, pad = is_v ? a.pad_vdim : a.pad_dim;
  const int chan0 = is_q ? head * a.dim : is_v ? (a.heads + a.kv_heads) * a.dim + kvh * a.vdim : (a.heads + kvh) * a.dim;
  float y[TT][4];
#pragma unroll
  for (int t = 0; t < TT; ++t)
#pragma unroll
    for (int v = 0; v < 4; ++v) y[t][v] = 0.0f;
  if (valid && l.e0 < dim) conv_rows<T, 4, 4, TT>(src, cr, row0, n, chan0 + l.e0, true, y);
  if (!is_v) {
    float ss[TT];
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      float other[4];
      ss[t] = 0.0f;
#pragma unroll
      for (int v = 0; v < 4; ++v) other[v] = __shfl_sync(0xffffffffu, y[t][v], l.partner);
#pragma unroll
      for (int v = 0; v < 4; ++v) {
        y[t][v] = fmaf(y[t][v], f.cs[t][v], other[v] * f.sn[t][v]);
        ss[t] = fmaf(y[t][v], y[t][v], ss[t]);      // 0 past dim
      }
    }
    if constexpr (TT == 4) {
      warp_sum4(ss);
    } else {
#pragma unroll
      for (int t = 0; t < TT; ++t) ss[t] = warp_sum(ss[t]);
    }
    const float inv_dim = 1.0f / static_cast<float>(a.dim);
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      const float r = rsqrtf(ss[t] * inv_dim + a.eps);
#pragma unroll
      for (int v = 0; v < 4; ++v) y[t][v] *= r;
    }
  }
  if (is_q) {
    T* dst = static_cast<T*>(a.q_out) + (static_cast<int64_t>(row0) * a.heads + head) * pad + l.e0;
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      if (t < n) {
        if (l.e0 < pad) store_f32<4>(dst, y[t]);
        for (int e = 128; e + l.lane < pad; e += 32) { const float z[1] = {0.0f}; store_f32<1>(dst - l.e0 + e + l.lane, z); }
      }
      dst += static_cast<int64_t>(a.heads) * pad;
    }
  } else if (l.e0 < dim) {
    T* cache = static_cast<T*>(is_v ? a.v_cache : a.k_cache) + static_cast<int64_t>(kvh) * a.page_size * pad + l.e0;
#pragma unroll
    for (int t = 0; t < TT; ++t)
      if (f.cell[t] >= 0) store_f32<4>(cache + static_cast<int64_t>(f.cell[t]) * pad, y[t]);
  }
}

template <typename T, int TT>
__global__ void __launch_bounds__(kWarps * 32, 3) conv_qkv_rows_kernel(const B2ConvQkvArgs a, const B2SeqRows sq, Status* status) {
  ptx::grid_dep_sync();
  const int n_heads = a.heads + 2 * a.kv_heads;
  const int channels = (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim;
  const ConvSource<T> src{static_cast<const T*>(a.proj), a.ld, a.conv_w, static_cast<T*>(a.conv_state), a.taps, channels, sq.banks};
  RowLane l;
  l.lane = threadIdx.x & 31;
  l.e0 = l.lane * 4;
  l.half = a.rot >> 1;
  l.turns = l.e0 < a.rot;
  l.lo = l.e0 < l.half;
  l.partner = l.turns ? (l.lo ? l.lane + l.half / 4 : l.lane - l.half / 4) : l.lane;
  const int64_t units = static_cast<int64_t>((sq.rows + TT - 1) / TT) * n_heads;
  const int64_t w = static_cast<int64_t>(blockIdx.x) * kWarps + (threadIdx.x >> 5), n_warps = static_cast<int64_t>(gridDim.x) * kWarps;
  int64_t left = units * (w + 1) / n_warps - units * w / n_warps;
  int tile = static_cast<int>(units * w / n_warps / n_heads), head = static_cast<int>(units * w / n_warps % n_heads);
  const auto place = [&](int row, ConvRow& cr) {
    const int seq = sq.row_seq[row];
    return seq >= 0 && B2_ASSERT(status, seq < sq.seqs, kSiteKvIndex, seq, sq.seqs) && cr.load(sq, seq, row, sq.banks, status);
  };
  for (; left > 0; ++tile, head = 0) {
    const int row0 = tile * TT, rows = min(TT, sq.rows - row0);
    const int stop = head + static_cast<int>(min(left, static_cast<int64_t>(n_heads - head)));      // this warp's heads of the tile
    left -= stop - head;
    ConvRow cr;
    const bool valid = place(row0, cr);
    if (TT == 1 || (valid && cr.end - row0 >= rows)) {
      RowFactors<TT> f;
      f.load(a, l, row0, rows, valid, status);
      for (; head < stop; ++head) conv_head<T, TT>(a, src, cr, valid, row0, rows, head, l, f);
    } else {
      for (int r = row0; r < row0 + rows; ++r) {
        const bool ok = place(r, cr);
        RowFactors<1> f;
        f.load(a, l, r, 1, ok, status);
        for (int h = head; h < stop; ++h) conv_head<T, 1>(a, src, cr, ok, r, 1, h, l, f);
      }
    }
  }
}

template <typename T>
int launch_conv_qkv_rows(const B2ConvQkvArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  const int n_heads = a.heads + 2 * a.kv_heads;
  const bool small = static_cast<int64_t>((s.rows + 3) / 4) * n_heads < 2 * kNumSMs * kWarps;      // one row at a time then
  const int64_t units = static_cast<int64_t>(small ? s.rows : (s.rows + 3) / 4) * n_heads, ctas = (units + kWarps - 1) / kWarps;
  const int grid = static_cast<int>(ctas < 3 * kNumSMs ? ctas : 3 * kNumSMs);
  if (small) launch_pdl(conv_qkv_rows_kernel<T, 1>, dim3(grid), dim3(kWarps * 32), 0, stream, a, s, status);
  else launch_pdl(conv_qkv_rows_kernel<T, 4>, dim3(grid), dim3(kWarps * 32), 0, stream, a, s, status);
  return last_launch_rc();
}

template <typename T, int VEC, int NJ, int TAPS>
int launch_conv_qkv(const B2ConvQkvArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  const int groups = (a.heads + 2 * a.kv_heads + kWarps - 1) / kWarps;
  // rows of one warp share the convolution's window; a small step wants one warp per row
  constexpr int kRows = TAPS == 0 ? 2 : 4;
  if ((s.rows + kRows - 1) / kRows * groups < 2 * kNumSMs)
    launch_pdl(conv_qkv_kernel<T, VEC, NJ, TAPS, 1>, dim3(s.rows, groups), dim3(kWarps * 32), 0, stream, a, s, status);
  else
    launch_pdl(conv_qkv_kernel<T, VEC, NJ, TAPS, kRows>, dim3((s.rows + kRows - 1) / kRows, groups), dim3(kWarps * 32), 0, stream, a, s, status);
  return last_launch_rc();
}

template <typename T>
int dispatch_conv_qkv(const B2ConvQkvArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  const bool kv = a.kv_heads > 0;
  const int d = kv && a.vdim > a.dim ? a.vdim : a.dim;
  const auto all = [&](int m) { return a.dim % m == 0 && (!kv || (a.vdim % m == 0 && a.pad_vdim % m == 0)) && a.ld % m == 0 && a.pad_dim % m == 0; };
  if (a.taps == 4 && all(4)) {
    if (d <= 128 && a.rot % 8 == 0) return launch_conv_qkv_rows<T>(a, s, status, stream);
    if (d <= 128) return launch_conv_qkv<T, 4, 1, 4>(a, s, status, stream);
    return launch_conv_qkv<T, 4, 2, 4>(a, s, status, stream);
  }
  if (all(2)) {
    if (d <= 128) return launch_conv_qkv<T, 2, 2, 0>(a, s, status, stream);
    return launch_conv_qkv<T, 2, 4, 0>(a, s, status, stream);
  }
  return launch_conv_qkv<T, 1, 8, 0>(a, s, status, stream);
}

// A thread's channels over a few rows of one sequence.
template <typename T, int VEC, int TAPS, int TT>
__global__ void __launch_bounds__(128) conv_silu_kernel(const B2ConvSiluArgs a, const B2SeqRows sq, Status* status) {
  ptx::grid_dep_sync();
  int tile = static_cast<int>(blockIdx.x);
  const int seq = find_tile(sq, 0, sq.seqs, TT, tile);
  if (seq < 0) return;
  const int row0 = sq.seq_rows[2 * seq] + tile * TT, c = static_cast<int>(blockIdx.y * 128 + threadIdx.x) * VEC;
  ConvRow cr;
  if (!cr.load(sq, seq, row0, sq.banks, status) || c >= a.channels) return;
  const ConvSource<T> src{static_cast<const T*>(a.proj), a.ld, a.conv_w, static_cast<T*>(a.conv_state), a.taps, a.channels, sq.banks};
  const int n = min(TT, cr.end - row0);
  float y[TT][VEC], b[VEC] = {};
  conv_rows<T, VEC, TAPS, TT>(src, cr, row0, n, c, true, y);
  if (a.bias != nullptr) load_f32<VEC>(a.bias + c, b);
#pragma unroll
  for (int t = 0; t < TT; ++t) {
    if (t >= n) break;
#pragma unroll
    for (int i = 0; i < VEC; ++i) y[t][i] = ptx::silu(y[t][i] + b[i]);
    store_f32<VEC>(static_cast<T*>(a.out) + static_cast<int64_t>(row0 + t) * a.ld_out + c, y[t]);
  }
}

template <typename T, int VEC, int TAPS>
int launch_conv_silu(const B2ConvSiluArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  constexpr int kRows = 8;
  const unsigned blocks = (a.channels + 128 * VEC - 1) / (128 * VEC);
  if (s.rows <= s.seqs) launch_pdl(conv_silu_kernel<T, VEC, TAPS, 1>, dim3(s.rows, blocks), dim3(128), 0, stream, a, s, status);
  else launch_pdl(conv_silu_kernel<T, VEC, TAPS, kRows>, dim3(s.rows / kRows + s.seqs, blocks), dim3(128), 0, stream, a, s, status);
  return last_launch_rc();
}

template <typename T>
int dispatch_conv_silu(const B2ConvSiluArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  if (a.channels % 4 == 0 && a.ld % 4 == 0 && a.ld_out % 4 == 0 && reinterpret_cast<uintptr_t>(a.proj) % (4 * sizeof(T)) == 0 &&
      reinterpret_cast<uintptr_t>(a.out) % (4 * sizeof(T)) == 0) {
    switch (a.taps) {
      case 2: return launch_conv_silu<T, 4, 2>(a, s, status, stream);
      case 3: return launch_conv_silu<T, 4, 3>(a, s, status, stream);
      case 4: return launch_conv_silu<T, 4, 4>(a, s, status, stream);
      default: return launch_conv_silu<T, 4, 0>(a, s, status, stream);
    }
  }
  return launch_conv_silu<T, 1, 0>(a, s, status, stream);
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_conv_silu(const B2ConvSiluArgs* a, const B2SeqRows* s, int f32, Status* status, cudaStream_t stream) {
  if (s->rows <= 0) return 0;
  if (a->channels <= 0 || a->taps < 1 || (a->taps > 1 && a->conv_state == nullptr) || a->out == nullptr || a->ld < a->channels || a->ld_out < a->channels)
    return -kBadArgument;
  return f32 ? dispatch_conv_silu<float>(*a, *s, status, stream) : dispatch_conv_silu<__nv_bfloat16>(*a, *s, status, stream);
}

extern "C" int b2_conv_qkv(const B2ConvQkvArgs* a, const B2SeqRows* s, int f32, Status* status, cudaStream_t stream) {
  if (s->rows <= 0) return 0;
  if (a->heads <= 0 || a->kv_heads < 0 || a->dim <= 0 || a->dim > kMaxHead || a->vdim > kMaxHead || a->pad_dim < a->dim || a->rot % 2 != 0 ||
      a->rot > a->dim || a->taps < 1 || (a->taps > 1 && a->conv_state == nullptr) || a->q_out == nullptr || (a->rot > 0 && a->cos_sin == nullptr))
    return -kBadArgument;
  if (a->kv_heads > 0 && (a->k_cache == nullptr || a->v_cache == nullptr || a->slots == nullptr || a->pad_vdim < a->vdim || a->page_size <= 0 || a->num_slots * a->kv_heads > 0x7fffffff ||
                          a->heads % a->kv_heads != 0))
    return -kBadArgument;
  return f32 ? dispatch_conv_qkv<float>(*a, *s, status, stream) : dispatch_conv_qkv<__nv_bfloat16>(*a, *s, status, stream);
}
