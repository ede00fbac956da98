// Attention front end of layers that normalise whole projections: biases, one RMS norm over all q columns of a row and one over
// its k columns, rotary embedding, scatter of k and v into the paged cache. One CTA per token row; the row's q and k wait in
// shared memory, in f32, for the two sums and for their rotation partners.
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

template <typename T, int VEC>
__global__ void __launch_bounds__(256) norm_qkv_kernel(const B2NormQkvArgs a, Status* status) {
  ptx::grid_dep_sync();
  extern __shared__ __align__(16) float row_sm[];
  __shared__ float scratch[33];
  const int64_t row = blockIdx.x;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim, half = a.rot >> 1;
  const T* src = static_cast<const T*>(a.proj) + row * a.ld;
  const int64_t slot = a.slots[row];
  const bool cached = slot >= 0 && B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots);
  // cache row of head 0; the heads of a page lie page_size rows apart
  const int64_t cell = cached ? slot / a.page_size * a.kv_heads * a.page_size + slot % a.page_size : 0;
  int pos = a.positions[row];
  if (!B2_ASSERT(status, pos >= 0 && (pos < a.max_pos || a.rot == 0), kSiteKvIndex, pos, a.max_pos)) pos = 0;
  const float* cs = a.cos_sin + static_cast<int64_t>(pos) * a.rot;
  float sq = 0.0f, sk = 0.0f;
  for (int c = threadIdx.x * VEC; c < nq + nk; c += blockDim.x * VEC) {      // VEC divides dim: a vector lies in one head
    float v[VEC], b[VEC], s = 0.0f;
    load_f32<VEC>(src + c, v);
    load_f32<VEC>(a.bias + c, b);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      v[i] += b[i];
      s = fmaf(v[i], v[i], s);
    }
    if (c < nq) sq += s;
    else sk += s;
    store_f32<VEC>(row_sm + c, v);
  }
  if (cached)
    for (int c = threadIdx.x * VEC; c < nv; c += blockDim.x * VEC) {
      float v[VEC], b[VEC];
      load_f32<VEC>(src + nq + nk + c, v);
      load_f32<VEC>(a.bias + nq + nk + c, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] += b[i];
      const int h = c / a.vdim;
      store_f32<VEC>(static_cast<T*>(a.v_cache) + (cell + static_cast<int64_t>(h) * a.page_size) * a.pad_vdim + c - h * a.vdim, v);
    }
  const float rq = 1.0f / sqrtf(block_sum(sq, scratch) / static_cast<float>(nq) + a.eps);
  const float rk = 1.0f / sqrtf(block_sum(sk, scratch) / static_cast<float>(nk) + a.eps);      // its barriers also publish row_sm
  for (int c = threadIdx.x * VEC; c < nq + nk; c += blockDim.x * VEC) {
    const bool is_q = c < nq;
    if (!is_q && !cached) break;
    const int h = (is_q ? c : c - nq) / a.dim, e0 = (is_q ? c : c - nq) - h * a.dim;
    const float r = is_q ? rq : rk;
    const float* w = is_q ? a.q_norm : a.k_norm - nq;      // indexed by c
    float v[VEC], g[VEC];
    load_f32<VEC>(row_sm + c, v);
    load_f32<VEC>(w + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] *= r * g[i];
    if (e0 < a.rot) {
      if (VEC > 1 && half % VEC == 0) {      // a vector lies on one side of the rotated span
        const bool lo = e0 < half;
        const int other = lo ? c + half : c - half;
        float o[VEC], og[VEC], cv[VEC], sv[VEC];
        load_f32<VEC>(row_sm + other, o);
        load_f32<VEC>(w + other, og);
        load_f32<VEC>(cs + (lo ? e0 : e0 - half), cv);
        load_f32<VEC>(cs + half + (lo ? e0 : e0 - half), sv);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = v[i] * cv[i] + (lo ? -1.0f : 1.0f) * (o[i] * (r * og[i])) * sv[i];
      } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const int e = e0 + i;
          if (e >= a.rot) continue;
          const bool lo = e < half;
          const int other = lo ? c + i + half : c + i - half, p = lo ? e : e - half;
          v[i] = v[i] * cs[p] + (lo ? -1.0f : 1.0f) * (row_sm[other] * (r * w[other])) * cs[half + p];
        }
      }
    }
    T* dst = is_q ? static_cast<T*>(a.q_out) + (row * a.heads + h) * a.pad_dim
                  : static_cast<T*>(a.k_cache) + (cell + static_cast<int64_t>(h) * a.page_size) * a.pad_dim;
    store_f32<VEC>(dst + e0, v);
  }
  // queries are zero past `dim`; cache rows are from the start
  const int gap = a.pad_dim - a.dim;
  for (int i = threadIdx.x; i < a.heads * gap; i += blockDim.x) {
    const float z[1] = {0.0f};
    store_f32<1>(static_cast<T*>(a.q_out) + (row * a.heads + i / gap) * a.pad_dim + a.dim + i % gap, z);
  }
}

template <typename T, int VEC>
int launch_norm_qkv(const B2NormQkvArgs& a, Status* status, cudaStream_t stream) {
  const int cols = (a.heads + a.kv_heads) * a.dim, smem = cols * 4;
  static DeviceOnce attr_once;
  if (smem > 40 * 1024)
    if (const int rc = attr_once.max_smem(norm_qkv_kernel<T, VEC>, 200 * 1024)) return rc;
  const int vecs = (cols + VEC - 1) / VEC;
  const int threads = vecs >= 256 ? 256 : (vecs + 31) / 32 * 32;
  launch_pdl(norm_qkv_kernel<T, VEC>, dim3(a.rows), dim3(threads), smem, stream, a, status);
  return last_launch_rc();
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_norm_qkv(const B2NormQkvArgs* a, int f32, Status* status, cudaStream_t stream) {
  if (a->rows <= 0) return 0;
  if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->dim <= 0 || a->vdim <= 0 || a->pad_dim < a->dim || a->pad_vdim < a->vdim ||
      a->rot < 0 || a->rot % 2 != 0 || a->rot > a->dim || a->page_size <= 0 || (a->rot > 0 && a->cos_sin == nullptr) ||
      static_cast<int64_t>(a->heads + a->kv_heads) * a->dim > 50000)
    return -kBadArgument;
  // every vector access must be aligned: rows, heads, caches, and the table's two halves
  const bool v4 = a->dim % 4 == 0 && a->vdim % 4 == 0 && a->pad_dim % 4 == 0 && a->pad_vdim % 4 == 0 && a->ld % 4 == 0 && reinterpret_cast<uintptr_t>(a->proj) % 16 == 0;
  if (f32) return v4 ? launch_norm_qkv<float, 4>(*a, status, stream) : launch_norm_qkv<float, 1>(*a, status, stream);
  return v4 ? launch_norm_qkv<__nv_bfloat16, 4>(*a, status, stream) : launch_norm_qkv<__nv_bfloat16, 1>(*a, status, stream);
}
