// Attention front end of layers with short convolutions: causal convolution over time on every q, k and v channel, rotary
// embedding, RMS norm of the q and k heads, scatter of k and v into the paged cache. One warp owns one head and a few
// consecutive rows. What the convolution needs from before the step comes from the sequence's state bank; the step's last
// taps - 1 projected rows go to its other bank, so no warp reads what another one of the same launch writes.
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/short_conv.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kMaxHead = 256;
constexpr int kWarps = 8;

template <typename T, int VEC, int NJ>
__global__ void __launch_bounds__(kWarps * 32) conv_qkv_kernel(const B2ConvQkvArgs a, const B2SeqRows sq, int rows_per_warp, Status* status) {
  ptx::grid_dep_sync();
  __shared__ float head_sm[kWarps][kMaxHead];
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
  const int row_end = min(sq.rows, static_cast<int>(blockIdx.x + 1) * rows_per_warp);
  for (int row = blockIdx.x * rows_per_warp; row < row_end; ++row) {
    const int seq = sq.row_seq[row];
    T* q_dst = static_cast<T*>(a.q_out) + static_cast<int64_t>(row) * a.heads * a.pad_dim + static_cast<int64_t>(head) * a.pad_dim;
    if (seq < 0 || !B2_ASSERT(status, seq < sq.seqs, kSiteKvIndex, seq, sq.seqs)) {
      if (is_q)
        for (int e = lane; e < pad; e += 32) { const float z[1] = {0.0f}; store_f32<1>(q_dst + e, z); }
      continue;
    }
    ConvRow cr;
    if (!cr.load(sq, seq, row, sq.banks, status)) continue;
    float val[NJ][VEC];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int e = (lane + 32 * j) * VEC;
      if (e < dim) {
        src.template apply<VEC>(cr, row, chan0 + e, val[j]);
        src.template save<VEC>(cr, row, chan0 + e);
      } else {
#pragma unroll
        for (int v = 0; v < VEC; ++v) val[j][v] = 0.0f;
      }
    }
    if (!is_v) {
      // rotate pairs (i, i + rot / 2), then divide by the root mean square of the head
      int pos = a.positions[row];
      if (!B2_ASSERT(status, pos >= 0 && pos < a.max_pos, kSiteKvIndex, pos, a.max_pos)) pos = 0;
      const float* cs = a.cos_sin + static_cast<int64_t>(pos) * a.rot;
      __syncwarp();
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int e = (lane + 32 * j) * VEC;
        if (e < dim) store_f32<VEC>(hs + e, val[j]);
      }
      __syncwarp();
      float ss = 0.0f;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          const int e = (lane + 32 * j) * VEC + v;
          if (e < half) val[j][v] = val[j][v] * cs[e] - hs[e + half] * cs[half + e];
          else if (e < a.rot) val[j][v] = val[j][v] * cs[e - half] + hs[e - half] * cs[e];
          ss = fmaf(val[j][v], val[j][v], ss);      // 0 past dim
        }
      }
      ss = warp_sum(ss);
      const float r = 1.0f / sqrtf(ss / static_cast<float>(dim) + a.eps);
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int v = 0; v < VEC; ++v) val[j][v] *= r;
    }
    T* dst = q_dst;
    int lim = pad;          // queries: zeros up to the padded size; cache rows are zero there from the start
    if (!is_q) {
      const int64_t slot = a.slots[row];
      if (slot < 0 || !B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots)) continue;
      T* cache = static_cast<T*>(is_v ? a.v_cache : a.k_cache);
      dst = cache + ((slot / a.page_size * a.kv_heads + kvh) * a.page_size + slot % a.page_size) * pad;
      lim = dim;
    }
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int e = (lane + 32 * j) * VEC;
      if (e < lim) store_f32<VEC>(dst + e, val[j]);
    }
    if (is_q)
      for (int e = 32 * NJ * VEC + lane; e < pad; e += 32) { const float z[1] = {0.0f}; store_f32<1>(dst + e, z); }
  }
}

template <typename T, int VEC, int NJ>
int launch_conv_qkv(const B2ConvQkvArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  const int groups = (a.heads + 2 * a.kv_heads + kWarps - 1) / kWarps;
  // consecutive rows of one warp share the convolution's history through L1, but a small step wants one warp per row
  int rpw = 8;
  while (rpw > 1 && (s.rows + rpw - 1) / rpw * groups < 4 * kNumSMs) rpw >>= 1;
  launch_pdl(conv_qkv_kernel<T, VEC, NJ>, dim3((s.rows + rpw - 1) / rpw, groups), dim3(kWarps * 32), 0, stream, a, s, rpw, status);
  return last_launch_rc();
}

template <typename T>
int dispatch_conv_qkv(const B2ConvQkvArgs& a, const B2SeqRows& s, Status* status, cudaStream_t stream) {
  const int d = a.dim > a.vdim && a.kv_heads > 0 ? a.dim : (a.kv_heads > 0 ? a.vdim : a.dim);
  const bool even = a.dim % 2 == 0 && (a.kv_heads == 0 || a.vdim % 2 == 0) && a.ld % 2 == 0 && a.pad_dim % 2 == 0 && a.pad_vdim % 2 == 0;
  if (!even) return launch_conv_qkv<T, 1, 8>(a, s, status, stream);
  if (d <= 64) return launch_conv_qkv<T, 2, 1>(a, s, status, stream);
  if (d <= 128) return launch_conv_qkv<T, 2, 2>(a, s, status, stream);
  return launch_conv_qkv<T, 2, 4>(a, s, status, stream);
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_conv_qkv(const B2ConvQkvArgs* a, const B2SeqRows* s, int f32, Status* status, cudaStream_t stream) {
  if (s->rows <= 0) return 0;
  if (a->heads <= 0 || a->kv_heads < 0 || a->dim <= 0 || a->dim > kMaxHead || a->vdim > kMaxHead || a->pad_dim < a->dim || a->rot % 2 != 0 ||
      a->rot > a->dim || a->taps < 1 || (a->taps > 1 && a->conv_state == nullptr) || a->q_out == nullptr || (a->rot > 0 && a->cos_sin == nullptr))
    return -kBadArgument;
  if (a->kv_heads > 0 && (a->k_cache == nullptr || a->v_cache == nullptr || a->slots == nullptr || a->pad_vdim < a->vdim || a->page_size <= 0 ||
                          a->heads % a->kv_heads != 0))
    return -kBadArgument;
  return f32 ? dispatch_conv_qkv<float>(*a, *s, status, stream) : dispatch_conv_qkv<__nv_bfloat16>(*a, *s, status, stream);
}
