// Hyper-connections: the residual is `streams` f32 copies of the row, mixed by small learned matrices around every
// sublayer. One kernel does everything between two sublayers: add the finished sublayer's output into all streams
// (each from the old ones), read the next sublayer's input off them, RMS-normalise it. One CTA per token row.
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

template <typename T, int S, int VEC>
__global__ void hyper_norm_kernel(const B2HyperArgs a, Status* status) {
  ptx::grid_dep_sync();
  extern __shared__ float u_sm[];    // the sublayer input of this row; every thread touches its own columns only
  __shared__ float scratch[33];
  int64_t row = blockIdx.x;
  if (a.rows_index != nullptr) {
    row = a.rows_index[blockIdx.x];
    if (!B2_ASSERT(status, row >= 0 && row < a.rows, kSiteKvIndex, row, a.rows)) return;   // uniform per CTA
  }
  float in[S], out[S], mix[S][S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    in[s] = a.in != nullptr ? a.in[s] : 1.0f;
    out[s] = a.y != nullptr ? a.out[s] : 0.0f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = a.y != nullptr ? a.mix[s * S + t] : (s == t ? 1.0f : 0.0f);
  }
  const int W = a.width;
  float* x = a.x + row * S * W;
  const T* y = a.y != nullptr ? static_cast<const T*>(a.y) + row * W : nullptr;
  const T* emb = nullptr;
  if (a.ids != nullptr) {
    const int64_t id = a.ids[row];
    if (B2_ASSERT(status, id >= 0 && id < a.vocab, kSiteKvIndex, id, a.vocab)) emb = static_cast<const T*>(a.embed) + id * W;
  }
  float ss = 0.0f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float old[S][VEC], u[VEC];
    if (a.ids != nullptr) {
      float e[VEC] = {};
      if (emb != nullptr) load_f32<VEC>(emb + c, e);
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int v = 0; v < VEC; ++v) old[s][v] = e[v] * a.embed_scale;
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) load_f32<VEC>(x + static_cast<int64_t>(s) * W + c, old[s]);
    }
    float yv[VEC] = {};
    if (y != nullptr) load_f32<VEC>(y + c, yv);
#pragma unroll
    for (int v = 0; v < VEC; ++v) u[v] = 0.0f;
#pragma unroll
    for (int t = 0; t < S; ++t) {
      float n[VEC];
      if (y != nullptr) {
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          n[v] = out[t] * yv[v];
#pragma unroll
          for (int s = 0; s < S; ++s) n[v] = fmaf(mix[s][t], old[s][v], n[v]);
        }
      } else {
#pragma unroll
        for (int v = 0; v < VEC; ++v) n[v] = old[t][v];
      }
      if (a.store) store_f32<VEC>(x + static_cast<int64_t>(t) * W + c, n);
#pragma unroll
      for (int v = 0; v < VEC; ++v) u[v] = fmaf(in[t], n[v], u[v]);
    }
#pragma unroll
    for (int v = 0; v < VEC; ++v) ss = fmaf(u[v], u[v], ss);
    store_f32<VEC>(u_sm + c, u);
  }
  ss = block_sum(ss, scratch);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(a.mean_width) + a.eps);
  T* h = static_cast<T*>(a.h) + static_cast<int64_t>(blockIdx.x) * W;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float u[VEC], w[VEC];
    load_f32<VEC>(u_sm + c, u);
    load_f32<VEC>(a.weight + c, w);
#pragma unroll
    for (int v = 0; v < VEC; ++v) u[v] = u[v] * r * w[v];
    store_f32<VEC>(h + c, u);
  }
}

template <typename T, int S, int VEC>
int launch_hyper(const B2HyperArgs& a, Status* status, cudaStream_t stream) {
  const int smem = a.width * 4;
  static DeviceOnce attr_once;
  if (smem > 40 * 1024)
    if (const int rc = attr_once.max_smem(hyper_norm_kernel<T, S, VEC>, 200 * 1024)) return rc;
  const int vecs = (a.width + VEC - 1) / VEC;
  const int threads = vecs >= 256 ? 256 : (vecs + 31) / 32 * 32;      // more threads per row would leave one row per SM
  launch_pdl(hyper_norm_kernel<T, S, VEC>, dim3(a.n_out), dim3(threads), smem, stream, a, status);
  return last_launch_rc();
}

template <typename T, int VEC>
int dispatch_hyper(const B2HyperArgs& a, Status* status, cudaStream_t stream) {
  switch (a.streams) {
    case 1: return launch_hyper<T, 1, VEC>(a, status, stream);
    case 2: return launch_hyper<T, 2, VEC>(a, status, stream);
    case 3: return launch_hyper<T, 3, VEC>(a, status, stream);
    case 4: return launch_hyper<T, 4, VEC>(a, status, stream);
    case 5: return launch_hyper<T, 5, VEC>(a, status, stream);
    case 6: return launch_hyper<T, 6, VEC>(a, status, stream);
    case 7: return launch_hyper<T, 7, VEC>(a, status, stream);
    case 8: return launch_hyper<T, 8, VEC>(a, status, stream);
    default: return -kBadArgument;
  }
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_hyper_norm(const B2HyperArgs* a, int f32, Status* status, cudaStream_t stream) {
  if (a->n_out <= 0) return 0;
  if (a->width <= 0 || a->width > 50000 || a->mean_width <= 0 || a->mean_width > a->width || a->x == nullptr || a->h == nullptr || a->weight == nullptr ||
      (a->y != nullptr && (a->mix == nullptr || a->out == nullptr)) || (a->ids != nullptr && a->embed == nullptr) ||
      (a->rows_index == nullptr && a->n_out != a->rows))
    return -kBadArgument;
  const bool v4 = a->width % 4 == 0;
  if (f32) return v4 ? dispatch_hyper<float, 4>(*a, status, stream) : dispatch_hyper<float, 1>(*a, status, stream);
  return v4 ? dispatch_hyper<__nv_bfloat16, 4>(*a, status, stream) : dispatch_hyper<__nv_bfloat16, 1>(*a, status, stream);
}
