// True 32-bit forms of the matrix product, gated linear units, row gather and paged attention, for models that run with f32
// activations on the GPU. Plain FMA throughout: no TF32 or other reduced-precision matrix mode.
#include <cstdint>
#include "b2/act.cuh"
#include "b2/api.h"
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kBM = 64, kBN = 64, kBK = 16;

// 64 x 64 tile, 256 threads of 4 x 4 outputs.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const B2GemmF32Args a) {
  ptx::grid_dep_sync();
  const int M = a.M, N = a.N, K = a.K;
  const int64_t ldx = a.ldx, ldw = a.ldw, col0 = static_cast<int64_t>(blockIdx.z) * N;
  const float* __restrict__ x = a.x + static_cast<int64_t>(blockIdx.z) * K;
  const float* __restrict__ w = a.w + col0 * ldw;
  __shared__ float xs[kBK][kBM + 4], ws[kBK][kBN + 4];
  const int m0 = blockIdx.y * kBM, n0 = blockIdx.x * kBN;
  const int tm = (threadIdx.x >> 4) * 4, tn = (threadIdx.x & 15) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kBK) {
    for (int i = threadIdx.x; i < kBM * kBK; i += 256) {
      const int r = i / kBK, c = i % kBK;
      xs[c][r] = m0 + r < M && k0 + c < K ? x[(m0 + r) * ldx + k0 + c] : 0.0f;
      ws[c][r] = n0 + r < N && k0 + c < K ? w[(n0 + r) * ldw + k0 + c] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kBK; ++k) {
      float xv[4], wv[4];
      load_f32<4>(&xs[k][tm], xv);
      load_f32<4>(&ws[k][tn], wv);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (m0 + tm + i < M && n0 + tn + j < N) {
        const int64_t m = m0 + tm + i, n = col0 + n0 + tn + j;
        float v = acc[i][j];
        if (a.epilogue == B2_EPI_RELU2) v = relu2(v);
        if (a.epilogue == B2_EPI_SOFTCAP) v = softcap(v, a.cap);
        if (a.gate != nullptr) v *= sigmoid_f32(a.gate[m * a.ld_gate + (a.gate_heads ? static_cast<int64_t>(blockIdx.z) : n)]);
        a.y[m * a.ldy + n] = v;
      }
}

__global__ void glu_f32_kernel(const float* __restrict__ gu, float* __restrict__ out, int64_t total, int ffn, B2EpiAct act) {
  ptx::grid_dep_sync();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const int64_t r = i / ffn;
  const int c = static_cast<int>(i % ffn);
  const float* p = gu + r * 2 * ffn + (c / 16) * 32 + c % 16;
  const float g = fminf(p[0], act.limit), u = fminf(fmaxf(p[16], -act.limit), act.limit);
  out[i] = g / (1.0f + expf(-act.alpha * g)) * (u + act.up_bias);
}

__global__ void gather_rows_f32_kernel(const float* __restrict__ src, const int64_t* __restrict__ index, float* __restrict__ out, int cols,
                                       int64_t rows_src, Status* status) {
  ptx::grid_dep_sync();
  const int64_t s = index[blockIdx.x];
  if (!B2_ASSERT(status, s >= 0 && s < rows_src, kSiteKvIndex, s, rows_src)) return;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) out[static_cast<int64_t>(blockIdx.x) * cols + c] = src[s * cols + c];
}

// One warp per (row, head): 32 keys at a time, a key per lane for the scores, a value column per lane for the output.
template <int kAttnMax>
__global__ void __launch_bounds__(128) attn_f32_kernel(const float* __restrict__ q, const float* __restrict__ kc, const float* __restrict__ vc,
                                                       float* __restrict__ out, const int32_t* __restrict__ row_seq,
                                                       const int32_t* __restrict__ positions, const int32_t* __restrict__ tables, int rows, int seqs,
                                                       int max_blocks, int n_q, int n_kv, int dim, int vdim, int64_t ld_v, int64_t ld_out, int page_size,
                                                       float scale, B2AttnMods mods, int64_t num_pages,
                                                       const float* __restrict__ gate, int64_t gate_stride, int gate_elems, Status* status) {
  ptx::grid_dep_sync();
  __shared__ float q_sm[4][kAttnMax];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t idx = static_cast<int64_t>(blockIdx.x) * 4 + warp;
  if (idx >= static_cast<int64_t>(rows) * n_q) return;
  const int row = static_cast<int>(idx / n_q), head = static_cast<int>(idx % n_q), kvh = head / (n_q / n_kv);
  float* dst = out + row * ld_out + static_cast<int64_t>(head) * vdim;
  const int seq = row_seq[row];
  const int ctx = seq >= 0 ? positions[row] + 1 : 0;
  if (seq < 0 || !B2_ASSERT(status, seq < seqs && ctx >= 1 && (ctx - 1) / page_size < max_blocks, kSiteKvIndex, seq, ctx)) {
    for (int c = lane; c < vdim; c += 32) dst[c] = 0.0f;
    return;
  }
  for (int i = lane; i < dim; i += 32) q_sm[warp][i] = q[(static_cast<int64_t>(row) * n_q + head) * dim + i];
  __syncwarp();
  const int32_t* table = tables + static_cast<int64_t>(seq) * max_blocks;
  auto slot_of = [&](int pos) -> int64_t {
    int64_t page = table[pos / page_size];
    if (!B2_ASSERT(status, page >= 0 && page < num_pages, kSiteKvIndex, page, num_pages)) page = 0;
    return (page * n_kv + kvh) * page_size + pos % page_size;
  };
  const int own = ctx - 1;
  int first = mods.window > 0 ? max(0, ctx - mods.window) : 0;
  if (mods.chunk > 0) first = max(first, own - own % mods.chunk);
  const float r1 = mods.distance != nullptr ? mods.distance[head] : 0.0f, r2 = mods.distance != nullptr ? mods.distance[n_q + head] : 0.0f;
  // the sink is a score of zero that has been seen already
  float m = mods.sink ? 0.0f : -INFINITY, l = mods.sink && lane == 0 ? 1.0f : 0.0f, o[kAttnMax / 32];
#pragma unroll
  for (int j = 0; j < kAttnMax / 32; ++j) o[j] = 0.0f;
  for (int p0 = first; p0 < ctx; p0 += 32) {
    const int pos = p0 + lane;
    int64_t slot = 0;
    float s = -INFINITY;
    if (pos < ctx) {
      slot = slot_of(pos);
      const float* k = kc + slot * dim;
      float dot = 0.0f;
      for (int i = 0; i < dim; ++i) dot = fmaf(q_sm[warp][i], k[i], dot);
      s = dot * scale;
      if (mods.softcap > 0.0f) s = softcap(s, mods.softcap);
      if (mods.distance != nullptr) s -= r1 * log1pf(r2 * static_cast<float>(own - pos));
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float corr = expf(m - m_new), p = pos < ctx ? expf(s - m_new) : 0.0f;
    m = m_new;
    l = l * corr + p;
#pragma unroll
    for (int j = 0; j < kAttnMax / 32; ++j) o[j] *= corr;
    const int n = min(32, ctx - p0);
    for (int t = 0; t < n; ++t) {
      const float pt = __shfl_sync(0xffffffffu, p, t);
      const float* v = vc + __shfl_sync(0xffffffffu, slot, t) * ld_v;
#pragma unroll
      for (int j = 0; j < kAttnMax / 32; ++j)
        if (lane + 32 * j < vdim) o[j] = fmaf(pt, v[lane + 32 * j], o[j]);
    }
  }
  float f = mods.out_scale / warp_sum(l);
  if (gate != nullptr && !gate_elems) f *= sigmoid_f32(gate[row * gate_stride + head]);
#pragma unroll
  for (int j = 0; j < kAttnMax / 32; ++j)
    if (lane + 32 * j < vdim) {
      const int c = lane + 32 * j;
      dst[c] = o[j] * f * (gate_elems ? sigmoid_f32(gate[row * gate_stride + static_cast<int64_t>(head) * vdim + c]) : 1.0f);
    }
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_gemm_f32(const B2GemmF32Args* a, cudaStream_t stream) {
  if (a->M <= 0 || a->N <= 0) return 0;
  if (a->K <= 0 || (a->M + kBM - 1) / kBM > 65535 || a->batch < 1 || a->batch > 65535 || (a->epilogue == B2_EPI_SOFTCAP && !(a->cap > 0.0f)) ||
      (a->epilogue != B2_EPI_NONE && a->epilogue != B2_EPI_RELU2 && a->epilogue != B2_EPI_SOFTCAP))
    return -kBadArgument;
  launch_pdl(gemm_f32_kernel, dim3((a->N + kBN - 1) / kBN, (a->M + kBM - 1) / kBM, a->batch), dim3(256), 0, stream, *a);
  return last_launch_rc();
}

extern "C" int b2_glu_f32(const float* gate_up, float* out, int64_t rows, int ffn, const B2EpiAct* act, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (ffn <= 0 || ffn % 16 != 0) return -kBadArgument;
  const int64_t total = rows * ffn;
  launch_pdl(glu_f32_kernel, dim3(static_cast<unsigned>((total + 255) / 256)), dim3(256), 0, stream, gate_up, out, total, ffn, act != nullptr ? *act : kPlainAct);
  return last_launch_rc();
}

extern "C" int b2_gather_rows_f32(const float* src, const int64_t* index, float* out, int rows_out, int cols, int64_t rows_src, Status* status,
                                  cudaStream_t stream) {
  if (rows_out <= 0) return 0;
  launch_pdl(gather_rows_f32_kernel, dim3(rows_out), dim3(128), 0, stream, src, index, out, cols, rows_src, status);
  return last_launch_rc();
}

extern "C" int b2_attn_f32(const float* q, const float* k_cache, const float* v_cache, float* out, const int32_t* row_seq, const int32_t* positions,
                           const int32_t* block_tables, int rows, int seqs, int max_blocks, int n_q, int n_kv, int dim, int vdim, int64_t ld_v, int64_t ld_out,
                           int page_size, float scale, const B2AttnMods* mods, int64_t num_pages, const float* gate, int64_t gate_stride,
                           int gate_elems, Status* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (n_kv <= 0 || n_q % n_kv != 0 || dim <= 0 || dim > 1152 || vdim <= 0 || vdim > 1152 || ld_v < vdim || ld_out < static_cast<int64_t>(n_q) * vdim ||
      page_size <= 0)
    return -kBadArgument;
  auto kern = dim <= 256 && vdim <= 256 ? attn_f32_kernel<256> : attn_f32_kernel<1152>;
  const int64_t warps = static_cast<int64_t>(rows) * n_q;
  launch_pdl(kern, dim3(static_cast<unsigned>((warps + 3) / 4)), dim3(128), 0, stream, q, k_cache, v_cache, out, row_seq, positions,
             block_tables, rows, seqs, max_blocks, n_q, n_kv, dim, vdim, ld_v, ld_out, page_size, scale, mods != nullptr ? *mods : B2AttnMods{0, 0, 0.0f, 1.0f, nullptr, 0},
             num_pages, gate, gate_stride, gate != nullptr ? gate_elems : 0, status);
  return last_launch_rc();
}
