// A plain residual kept in f32: one kernel between any two sublayers adds the finished one (a matrix product's rows, the
// weighted rows of a token's experts, a row with a gate, or several of them, scaled per channel) and RMS- or layer-normalises
// what the next one reads. The first
// call starts the stream from the embedding tables. One CTA per token row.
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kMaxTop = 32;

template <typename T, int VEC>
__global__ void residual_norm_kernel(const B2ResidualArgs a, Status* status) {
  ptx::grid_dep_sync();
  extern __shared__ float x_sm[];    // the row; every thread touches its own columns only
  __shared__ float scratch[33], e_w[kMaxTop];
  __shared__ int e_row[kMaxTop];
  int64_t row = blockIdx.x;
  if (a.rows_index != nullptr) {
    row = a.rows_index[blockIdx.x];
    if (!B2_ASSERT(status, row >= 0 && row < a.rows, kSiteKvIndex, row, a.rows)) return;   // uniform per CTA
  }
  if (a.experts != nullptr) {
    if (threadIdx.x < a.top) {
      const int slot = a.expert_slot[row * a.top + threadIdx.x];
      const bool ok = B2_ASSERT(status, slot >= (a.own != nullptr ? -1 : 0) && slot < a.expert_rows, kSiteEpCount, slot, a.expert_rows);
      e_row[threadIdx.x] = ok ? slot : 0;
      e_w[threadIdx.x] = !ok ? 0.0f : a.expert_w != nullptr ? a.expert_w[row * a.top + threadIdx.x] : 1.0f;
    }
    __syncthreads();
  }
  const int W = a.width;
  float* x = a.x + row * W;
  const T* y = a.y != nullptr ? static_cast<const T*>(a.y) + row * W : nullptr;
  const T *emb = nullptr, *big = nullptr;
  if (a.ids != nullptr) {
    const int64_t id = a.ids[row];
    if (B2_ASSERT(status, id >= 0 && id < a.vocab, kSiteKvIndex, id, a.vocab)) {
      emb = static_cast<const T*>(a.embed) + id * W;
      if (a.bigram != nullptr) {
        const int64_t prev = a.prev[row];
        const int64_t at = prev < 0 ? a.buckets : (prev * a.mul_prev + id * a.mul_cur) % a.buckets;
        if (B2_ASSERT(status, at >= 0 && at <= a.buckets, kSiteKvIndex, at, a.buckets)) big = static_cast<const T*>(a.bigram) + at * W;
      }
    }
  }
  const T* own = a.own != nullptr ? static_cast<const T*>(a.own) + row * W : nullptr;
  const T* gated = a.gated != nullptr ? static_cast<const T*>(a.gated) + row * W : nullptr;
  const float gate = gated != nullptr ? sigmoid_f32(a.gate[row * a.ld_gate]) : 0.0f;
  const bool fold = y != nullptr || a.experts != nullptr || gated != nullptr;
  float ss = 0.0f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC];
    if (a.ids != nullptr) {
      float e[VEC] = {}, b[VEC] = {};
      if (emb != nullptr) load_f32<VEC>(emb + c, e);
      if (big != nullptr) load_f32<VEC>(big + c, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = fmaf(e[i], a.embed_scale, b[i]);
      if (a.x0 != nullptr) store_f32<VEC>(static_cast<T*>(a.x0) + row * a.ld_x0 + c, v);
    } else {
      load_f32<VEC>(x + c, v);
    }
    if (fold) {
      float u[VEC] = {}, s[VEC];
      if (y != nullptr) load_f32<VEC>(y + c, u);
      if (a.experts != nullptr) {
        for (int j0 = 0; j0 < a.top; j0 += 4) {       // the rows of up to four experts are requested before the first is used
          float e[4][VEC];
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (j0 + j < a.top)
              load_f32<VEC>((e_row[j0 + j] < 0 ? own : static_cast<const T*>(a.experts) + static_cast<int64_t>(e_row[j0 + j]) * W) + c, e[j]);
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (j0 + j < a.top)
#pragma unroll
              for (int i = 0; i < VEC; ++i) u[i] = fmaf(e_w[j0 + j], e[j][i], u[i]);
        }
      }
      if (gated != nullptr) {
        float g[VEC];
        load_f32<VEC>(gated + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = fmaf(gate, g[i], u[i]);
      }
      if (a.y_scale != nullptr) {
        load_f32<VEC>(a.y_scale + c, s);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = fmaf(s[i], u[i], v[i]);
      } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] += u[i];
      }
    }
    if (a.store && (fold || a.ids != nullptr)) store_f32<VEC>(x + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = a.bias != nullptr ? ss + v[i] : fmaf(v[i], v[i], ss);
    store_f32<VEC>(x_sm + c, v);
  }
  T* h = static_cast<T*>(a.h) + static_cast<int64_t>(blockIdx.x) * a.ld_h;
  float r = 1.0f, mean = 0.0f;
  if (a.bias != nullptr) {      // layer norm: squares of the deviations in a second pass
    mean = block_sum(ss, scratch) / static_cast<float>(a.mean_width);
    ss = 0.0f;
    for (int c = threadIdx.x * VEC; c < a.mean_width; c += blockDim.x * VEC) {
      float v[VEC];
      load_f32<VEC>(x_sm + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i)
        if (c + i < a.mean_width) ss = fmaf(v[i] - mean, v[i] - mean, ss);
    }
  }
  if (a.weight != nullptr) r = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(a.mean_width) + a.eps);
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC], w[VEC];
    load_f32<VEC>(x_sm + c, v);
    if (a.weight != nullptr) {
      load_f32<VEC>(a.weight + c, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = (v[i] - mean) * r * w[i];
      if (a.bias != nullptr) {
        load_f32<VEC>(a.bias + c, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] += w[i];
      }
    }
    store_f32<VEC>(h + c, v);
  }
}

template <typename T, int VEC>
int launch_residual(const B2ResidualArgs& a, Status* status, cudaStream_t stream) {
  const int smem = a.width * 4;
  static DeviceOnce attr_once;
  if (smem > 40 * 1024)
    if (const int rc = attr_once.max_smem(residual_norm_kernel<T, VEC>, 200 * 1024)) return rc;
  const int vecs = (a.width + VEC - 1) / VEC;
  const int threads = vecs >= 256 ? 256 : (vecs + 31) / 32 * 32;
  launch_pdl(residual_norm_kernel<T, VEC>, dim3(a.n_out), dim3(threads), smem, stream, a, status);
  return last_launch_rc();
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_residual_norm(const B2ResidualArgs* a, int f32, Status* status, cudaStream_t stream) {
  if (a->n_out <= 0) return 0;
  if (a->width <= 0 || a->width > 50000 || a->mean_width <= 0 || a->mean_width > a->width || a->x == nullptr || a->h == nullptr ||
      (a->bias != nullptr && a->weight == nullptr) || (a->gated != nullptr && a->gate == nullptr) || (a->experts != nullptr && (a->expert_slot == nullptr || a->top < 1 || a->top > kMaxTop)) ||
      (a->ids != nullptr && a->embed == nullptr) || (a->bigram != nullptr && (a->prev == nullptr || a->buckets < 1)) ||
      (a->rows_index == nullptr && a->n_out != a->rows))
    return -kBadArgument;
  const bool v4 = a->width % 4 == 0 && a->ld_h % 4 == 0 && a->ld_x0 % 4 == 0;
  if (f32) return v4 ? launch_residual<float, 4>(*a, status, stream) : launch_residual<float, 1>(*a, status, stream);
  return v4 ? launch_residual<__nv_bfloat16, 4>(*a, status, stream) : launch_residual<__nv_bfloat16, 1>(*a, status, stream);
}
