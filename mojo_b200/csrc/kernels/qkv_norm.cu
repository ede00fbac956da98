// Attention front ends with norms. Over whole projections: biases, one RMS norm over all q columns of a row and one over
// its k columns, rotary embedding, scatter of k and v into the paged cache. One CTA per token row. Per head: one warp per
// (row, few heads).
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/short_conv.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

// The common case: a head is at most four columns per lane, and rotation partners lie whole lanes apart. A warp keeps its (up to
// HP) heads in registers, all of them requested at once.
template <typename T, int HP>
__global__ void __launch_bounds__(256) norm_qkv_heads_kernel(const B2NormQkvArgs a, Status* status) {
  ptx::grid_dep_sync();
  __shared__ float part[2][8];
  const int64_t row = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5, e0 = lane * 4;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, half = a.rot >> 1, n_heads = a.heads + a.kv_heads;
  const bool in_k = e0 < a.dim, in_v = e0 < a.vdim, turns = e0 < a.rot, lo = e0 < half;
  const T* src = static_cast<const T*>(a.proj) + row * a.ld;
  float v[HP][4], b[HP][4];
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    const int h = warp + i * n_warps, c = h * a.dim + e0;
#pragma unroll
    for (int j = 0; j < 4; ++j) v[i][j] = b[i][j] = 0.0f;
    if (h < n_heads && in_k) {
      load_f32<4>(src + c, v[i]);
      load_f32<4>(a.bias + c, b[i]);
    }
  }
  const int64_t slot = a.slots[row];
  const bool cached = slot >= 0 && B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots);
  // cache row of head 0; the heads of a page lie page_size rows apart (the host keeps slots below 2^31)
  const uint32_t page = cached ? static_cast<uint32_t>(slot) / static_cast<uint32_t>(a.page_size) : 0;
  const int64_t cell = cached ? static_cast<int64_t>(page) * a.kv_heads * a.page_size + (static_cast<uint32_t>(slot) - page * a.page_size) : 0;
  float cs[4] = {1.0f, 1.0f, 1.0f, 1.0f}, sn[4] = {0.0f, 0.0f, 0.0f, 0.0f};
  if (turns) {
    int pos = a.positions[row];
    if (!B2_ASSERT(status, pos >= 0 && pos < a.max_pos, kSiteKvIndex, pos, a.max_pos)) pos = 0;
    const float* at = a.cos_sin + static_cast<int64_t>(pos) * a.rot + (lo ? e0 : e0 - half);
    load_f32<4>(at, cs);
    load_f32<4>(at + half, sn);
    if (lo) {
#pragma unroll
      for (int j = 0; j < 4; ++j) sn[j] = -sn[j];
    }
  }
  const int partner = turns ? (lo ? lane + half / 4 : lane - half / 4) : lane;
  float sq = 0.0f, sk = 0.0f;
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    float s = 0.0f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      v[i][j] += b[i][j];
      s = fmaf(v[i][j], v[i][j], s);
    }
    if (warp + i * n_warps < a.heads) sq += s;
    else sk += s;
  }
  // the norm weights are on their way during the sums
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    const int h = warp + i * n_warps, c = h * a.dim + e0;
    if (h < n_heads && in_k) load_f32<4>(h < a.heads ? a.q_norm + c : a.k_norm + c - nq, b[i]);
  }
  if (cached)
    for (int h = warp; h < a.kv_heads; h += n_warps)
      if (in_v) {
        const int c = nq + nk + h * a.vdim + e0;
        float x[4], y[4];
        load_f32<4>(src + c, x);
        load_f32<4>(a.bias + c, y);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] += y[j];
        store_f32<4>(static_cast<T*>(a.v_cache) + (cell + static_cast<int64_t>(h) * a.page_size) * a.pad_vdim + e0, x);
      }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) {
    part[0][warp] = sq;
    part[1][warp] = sk;
  }
  __syncthreads();
  sq = sk = 0.0f;
  for (int w = 0; w < n_warps; ++w) {
    sq += part[0][w];
    sk += part[1][w];
  }
  const float rq = 1.0f / sqrtf(sq / static_cast<float>(nq) + a.eps), rk = 1.0f / sqrtf(sk / static_cast<float>(nk) + a.eps);
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    const int h = warp + i * n_warps;
    if (h >= n_heads) break;      // uniform per warp, as the next
    const bool is_q = h < a.heads;
    if (!is_q && !cached) break;
    const float r = is_q ? rq : rk;
    float o[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) v[i][j] *= r * b[i][j];
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] = __shfl_sync(0xffffffffu, v[i][j], partner);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[i][j] = fmaf(v[i][j], cs[j], o[j] * sn[j]);
    T* dst = is_q ? static_cast<T*>(a.q_out) + (row * a.heads + h) * a.pad_dim
                  : static_cast<T*>(a.k_cache) + (cell + static_cast<int64_t>(h - a.heads) * a.page_size) * a.pad_dim;
    // queries are zero past `dim` (as v is there); cache rows are from the start
    if (e0 < (is_q ? a.pad_dim : a.dim)) store_f32<4>(dst + e0, v[i]);
    if (is_q)
      for (int e = 128 + lane; e < a.pad_dim; e += 32) {
        const float z[1] = {0.0f};
        store_f32<1>(dst + e, z);
      }
  }
}

// Many rows of bf16, key and value heads of one size, a power of two: a thread takes NV vectors of eight columns, a head lies in
// neighbouring lanes of one warp. Persistent CTAs keep biases and norm weights in shared memory and request a row's values while
// they work on the one before.
template <int NV>
__global__ void __launch_bounds__(256, 3) norm_qkv_rows_kernel(const B2NormQkvArgs a, int log_dim, Status* status) {
  ptx::grid_dep_sync();
  extern __shared__ __align__(16) float par_sm[];      // biases of all columns, norm weights of q and k
  __shared__ float part[2][2][8];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, dim = 1 << log_dim;
  const int nq = a.heads << log_dim, nk = a.kv_heads << log_dim, cols = nq + 2 * nk, half = a.rot >> 1;
  float* w_sm = par_sm + cols;
  for (int c = threadIdx.x; c < cols; c += 256) {
    par_sm[c] = a.bias[c];
    if (c < nq + nk) w_sm[c] = c < nq ? a.q_norm[c] : a.k_norm[c - nq];
  }
  const int e0 = (lane * 8) & (dim - 1);      // the same in all of a thread's vectors: 2048 columns apart
  const bool turns = e0 < a.rot, lo = e0 < half;
  const int partner = turns ? (lo ? lane + half / 8 : lane - half / 8) : lane;
  const auto column = [&](int i) { return static_cast<int>(threadIdx.x + 256 * i) * 8; };
  uint4 next[NV];
  const auto request = [&](int64_t row) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      next[i] = make_uint4(0, 0, 0, 0);
      if (column(i) < cols) next[i] = ptx::ld_v4(static_cast<const __nv_bfloat16*>(a.proj) + row * a.ld + column(i));
    }
  };
  if (static_cast<int>(blockIdx.x) < a.rows) request(blockIdx.x);
  __syncthreads();
  int turn = 0;
  for (int64_t row = blockIdx.x; row < a.rows; row += gridDim.x, turn ^= 1) {
    const int64_t slot = a.slots[row];
    float cs[8], sn[8], v[NV][8], sq = 0.0f, sk = 0.0f;
    if (turns) {
      int pos = a.positions[row];
      if (!B2_ASSERT(status, pos >= 0 && pos < a.max_pos, kSiteKvIndex, pos, a.max_pos)) pos = 0;
      const float* at = a.cos_sin + static_cast<int64_t>(pos) * a.rot + (lo ? e0 : e0 - half);
#pragma unroll
      for (int j = 0; j < 8; j += 4) {
        load_f32<4>(at + j, *reinterpret_cast<float(*)[4]>(cs + j));
        load_f32<4>(at + half + j, *reinterpret_cast<float(*)[4]>(sn + j));
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      cs[j] = turns ? cs[j] : 1.0f;
      sn[j] = turns ? (lo ? -sn[j] : sn[j]) : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = column(i);
      float s = 0.0f;
      bf16x8_to_f32(next[i], v[i]);
      if (c < cols) {
#pragma unroll
        for (int j = 0; j < 8; j += 4) {
          float b[4];
          load_f32<4>(par_sm + c + j, b);
#pragma unroll
          for (int x = 0; x < 4; ++x) v[i][j + x] += b[x];
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) s = fmaf(v[i][j], v[i][j], s);
      if (c < nq) sq += s;
      else if (c < nq + nk) sk += s;
    }
    if (row + gridDim.x < a.rows) request(row + gridDim.x);
    const bool cached = slot >= 0 && B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots);
    // cache row of head 0; the heads of a page lie page_size rows apart (the host keeps slots below 2^31)
    const uint32_t page = cached ? static_cast<uint32_t>(slot) / static_cast<uint32_t>(a.page_size) : 0;
    const int64_t cell = cached ? static_cast<int64_t>(page) * a.kv_heads * a.page_size + (static_cast<uint32_t>(slot) - page * a.page_size) : 0;
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) {
      part[turn][0][warp] = sq;
      part[turn][1][warp] = sk;
    }
    __syncthreads();      // two sets of partial sums: one barrier a row is enough
    sq = sk = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      sq += part[turn][0][w];
      sk += part[turn][1][w];
    }
    const float rq = rsqrtf(sq / static_cast<float>(nq) + a.eps), rk = rsqrtf(sk / static_cast<float>(nk) + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = column(i);
      if (c < nq + nk) {
        const float r = c < nq ? rq : rk;
#pragma unroll
        for (int j = 0; j < 8; j += 4) {
          float w[4];
          load_f32<4>(w_sm + c + j, w);
#pragma unroll
          for (int x = 0; x < 4; ++x) v[i][j + x] *= r * w[x];
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float o = __shfl_sync(0xffffffffu, v[i][j], partner);
        if (c < nq + nk) v[i][j] = fmaf(v[i][j], cs[j], o * sn[j]);
      }
      const int h = c >> log_dim;
      __nv_bfloat16* dst = nullptr;
      if (c < nq) dst = static_cast<__nv_bfloat16*>(a.q_out) + (row * a.heads + h) * a.pad_dim;
      else if (cached && c < cols)
        dst = c < nq + nk ? static_cast<__nv_bfloat16*>(a.k_cache) + (cell + static_cast<int64_t>(h - a.heads) * a.page_size) * a.pad_dim
                          : static_cast<__nv_bfloat16*>(a.v_cache) + (cell + static_cast<int64_t>(h - a.heads - a.kv_heads) * a.page_size) * a.pad_vdim;
      if (dst != nullptr) ptx::st_v4(dst + e0, f32_to_bf16x8(v[i]));
    }
    // queries are zero past `dim`; cache rows are from the start
    const int gap = a.pad_dim - dim;
    for (int i = threadIdx.x * 8; i < a.heads * gap; i += 256 * 8)
      ptx::st_v4(static_cast<__nv_bfloat16*>(a.q_out) + (row * a.heads + i / gap) * a.pad_dim + dim + i % gap, make_uint4(0, 0, 0, 0));
  }
}

int launch_norm_qkv_rows(const B2NormQkvArgs& a, Status* status, cudaStream_t stream) {
  const int cols = (a.heads + 2 * a.kv_heads) * a.dim, nv = (cols + 2047) / 2048, smem = (cols + (a.heads + a.kv_heads) * a.dim) * 4;
  auto kern = nv == 1 ? norm_qkv_rows_kernel<1> : nv == 2 ? norm_qkv_rows_kernel<2> : nv == 3 ? norm_qkv_rows_kernel<3> : norm_qkv_rows_kernel<4>;
  static DeviceOnce attr_once[4];
  if (const int rc = attr_once[nv - 1].max_smem(kern, 72 * 1024)) return rc;
  int log_dim = 0;
  while ((1 << log_dim) < a.dim) ++log_dim;
  const int per_sm = (kMaxSmemPerCta - 4096) / (smem + 2048);
  launch_pdl(kern, dim3(kNumSMs * (per_sm < 3 ? per_sm : 3)), dim3(256), smem, stream, a, log_dim, status);
  return last_launch_rc();
}

// Any sizes: the row's q and k wait in shared memory, in f32, for the two sums and for their rotation partners. Warps take whole
// heads, lanes VEC columns at a time.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) norm_qkv_kernel(const B2NormQkvArgs a, Status* status) {
  ptx::grid_dep_sync();
  extern __shared__ __align__(16) float row_sm[];
  __shared__ float part[2][8];
  const int64_t row = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, half = a.rot >> 1, n_heads = a.heads + a.kv_heads;
  const T* src = static_cast<const T*>(a.proj) + row * a.ld;
  float sq = 0.0f, sk = 0.0f;
#pragma unroll 4
  for (int h = warp; h < n_heads; h += n_warps)
    for (int e = lane * VEC; e < a.dim; e += 32 * VEC) {
      const int c = h * a.dim + e;
      float v[VEC], b[VEC], s = 0.0f;
      load_f32<VEC>(src + c, v);
      load_f32<VEC>(a.bias + c, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        v[i] += b[i];
        s = fmaf(v[i], v[i], s);
      }
      if (h < a.heads) sq += s;
      else sk += s;
      store_f32<VEC>(row_sm + c, v);
    }
  const int64_t slot = a.slots[row];
  const bool cached = slot >= 0 && B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots);
  // cache row of head 0; the heads of a page lie page_size rows apart (the host keeps slots below 2^31)
  const uint32_t page = cached ? static_cast<uint32_t>(slot) / static_cast<uint32_t>(a.page_size) : 0;
  const int64_t cell = cached ? static_cast<int64_t>(page) * a.kv_heads * a.page_size + (static_cast<uint32_t>(slot) - page * a.page_size) : 0;
  int pos = a.positions[row];
  if (!B2_ASSERT(status, pos >= 0 && (pos < a.max_pos || a.rot == 0), kSiteKvIndex, pos, a.max_pos)) pos = 0;
  const float* cs = a.cos_sin + static_cast<int64_t>(pos) * a.rot;
  if (cached)
    for (int h = warp; h < a.kv_heads; h += n_warps)
      for (int e = lane * VEC; e < a.vdim; e += 32 * VEC) {
        const int c = nq + nk + h * a.vdim + e;
        float v[VEC], b[VEC];
        load_f32<VEC>(src + c, v);
        load_f32<VEC>(a.bias + c, b);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] += b[i];
        store_f32<VEC>(static_cast<T*>(a.v_cache) + (cell + static_cast<int64_t>(h) * a.page_size) * a.pad_vdim + e, v);
      }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) {
    part[0][warp] = sq;
    part[1][warp] = sk;
  }
  __syncthreads();      // also publishes row_sm
  sq = sk = 0.0f;
  for (int w = 0; w < n_warps; ++w) {
    sq += part[0][w];
    sk += part[1][w];
  }
  const float rq = 1.0f / sqrtf(sq / static_cast<float>(nq) + a.eps), rk = 1.0f / sqrtf(sk / static_cast<float>(nk) + a.eps);
#pragma unroll 2
  for (int h = warp; h < n_heads; h += n_warps) {
    const bool is_q = h < a.heads;
    if (!is_q && !cached) break;
    const float r = is_q ? rq : rk;
    const float* w = is_q ? a.q_norm : a.k_norm - nq;      // indexed by column of the row
    T* dst = is_q ? static_cast<T*>(a.q_out) + (row * a.heads + h) * a.pad_dim
                  : static_cast<T*>(a.k_cache) + (cell + static_cast<int64_t>(h - a.heads) * a.page_size) * a.pad_dim;
    for (int e0 = lane * VEC; e0 < a.dim; e0 += 32 * VEC) {
      const int c = h * a.dim + e0;
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
      store_f32<VEC>(dst + e0, v);
    }
    // queries are zero past `dim`; cache rows are from the start
    if (is_q)
      for (int e = a.dim + lane; e < a.pad_dim; e += 32) {
        const float z[1] = {0.0f};
        store_f32<1>(dst + e, z);
      }
  }
}

template <typename T>
int launch_norm_qkv_heads(const B2NormQkvArgs& a, Status* status, cudaStream_t stream) {
  const int n_heads = a.heads + a.kv_heads, threads = n_heads >= 8 ? 256 : n_heads * 32, per_warp = (n_heads + 7) / 8;
  auto kern = per_warp <= 1 ? norm_qkv_heads_kernel<T, 1> : per_warp <= 3 ? norm_qkv_heads_kernel<T, 3> : per_warp <= 5 ? norm_qkv_heads_kernel<T, 5>
                                                                                                        : norm_qkv_heads_kernel<T, 8>;
  launch_pdl(kern, dim3(a.rows), dim3(threads), 0, stream, a, status);
  return last_launch_rc();
}

template <typename T, int VEC>
int launch_norm_qkv(const B2NormQkvArgs& a, Status* status, cudaStream_t stream) {
  const int cols = (a.heads + a.kv_heads) * a.dim, smem = cols * 4;
  static DeviceOnce attr_once;
  if (smem > 40 * 1024)
    if (const int rc = attr_once.max_smem(norm_qkv_kernel<T, VEC>, 200 * 1024)) return rc;
  const int n_heads = a.heads + a.kv_heads, threads = n_heads >= 8 ? 256 : n_heads * 32;
  launch_pdl(norm_qkv_kernel<T, VEC>, dim3(a.rows), dim3(threads), smem, stream, a, status);
  return last_launch_rc();
}

// Warps take HP neighbouring heads of a row, all of them requested at once; a lane holds columns (lane + 32 j) * VEC.
template <typename T, int VEC, int NJ, int HP>
__global__ void __launch_bounds__(256) head_norm_qkv_kernel(const B2HeadNormArgs a, Status* status) {
  ptx::grid_dep_sync();
  const int n_heads = a.heads + 2 * a.kv_heads, runs = (n_heads + HP - 1) / HP, lane = threadIdx.x & 31;
  const int64_t idx = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5), row = idx / runs;
  if (row >= a.rows) return;
  const int h0 = static_cast<int>(idx % runs) * HP;
  const T* src = static_cast<const T*>(a.proj) + row * a.ld;
  const int64_t slot = a.slots[row];
  float v[HP][NJ][VEC], ss[HP];
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    const int h = h0 + i, kv = h - a.heads;
    const bool is_v = kv >= a.kv_heads;
    const int size = is_v ? a.vdim : a.dim, from = is_v ? a.v_off + (kv - a.kv_heads) * a.vdim : h * a.dim;
    ss[i] = 0.0f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = (lane + 32 * j) * VEC;
#pragma unroll
      for (int x = 0; x < VEC; ++x) v[i][j][x] = 0.0f;
      if (h < n_heads && c < size) load_f32<VEC>(src + from + c, v[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < HP; ++i) {
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
      for (int x = 0; x < VEC; ++x) ss[i] = fmaf(v[i][j][x], v[i][j][x], ss[i]);
  }
#pragma unroll
  for (int i = 0; i < HP; ++i) ss[i] = warp_sum(ss[i]);
  const bool cached = slot >= 0 && B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots);
  // cache row of head 0; the heads of a page lie page_size rows apart (the host keeps slots below 2^31)
  const uint32_t page = cached ? static_cast<uint32_t>(slot) / static_cast<uint32_t>(a.page_size) : 0;
  const int64_t cell = cached ? static_cast<int64_t>(page) * a.kv_heads * a.page_size + (static_cast<uint32_t>(slot) - page * a.page_size) : 0;
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    const int h = h0 + i, kv = h - a.heads;
    if (h >= n_heads || (kv >= 0 && !cached)) break;      // uniform per warp
    const bool is_q = kv < 0, is_v = kv >= a.kv_heads;
    T* dst = is_q ? static_cast<T*>(a.q_out) + (row * a.heads + h) * a.pad_dim
             : is_v ? static_cast<T*>(a.v_cache) + (cell + static_cast<int64_t>(kv - a.kv_heads) * a.page_size) * a.pad_vdim
                    : static_cast<T*>(a.k_cache) + (cell + static_cast<int64_t>(kv) * a.page_size) * a.pad_dim;
    const float* w = is_q ? a.q_norm : a.k_norm;
    const float r = 1.0f / sqrtf(ss[i] / static_cast<float>(a.dim) + a.eps);
    const int size = is_v ? a.vdim : a.dim;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = (lane + 32 * j) * VEC;
      if (!is_v && c < size) {
        float f[VEC];
        load_f32<VEC>(w + c, f);
#pragma unroll
        for (int x = 0; x < VEC; ++x) v[i][j][x] *= r * f[x];
      }
      // queries are zero past `dim` (as v is there); cache rows are from the start
      if (c < (is_q ? a.pad_dim : size)) store_f32<VEC>(dst + c, v[i][j]);
    }
  }
}

template <typename T, int VEC, int NJ, int HP>
int launch_head_norm(const B2HeadNormArgs& a, Status* status, cudaStream_t stream) {
  const int64_t warps = static_cast<int64_t>(a.rows) * ((a.heads + 2 * a.kv_heads + HP - 1) / HP);
  launch_pdl(head_norm_qkv_kernel<T, VEC, NJ, HP>, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, stream, a, status);
  return last_launch_rc();
}
template <typename T>
int dispatch_head_norm(const B2HeadNormArgs& a, Status* status, cudaStream_t stream) {
  const int m = a.pad_dim > a.pad_vdim ? a.pad_dim : a.pad_vdim;
  const bool v4 = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.v_off % 4 == 0 && a.pad_dim % 4 == 0 && a.pad_vdim % 4 == 0 && a.ld % 4 == 0 &&
                  reinterpret_cast<uintptr_t>(a.proj) % (4 * sizeof(T)) == 0;
  if (!v4) return launch_head_norm<T, 1, 8, 1>(a, status, stream);
  if (m > 128) return launch_head_norm<T, 4, 2, 2>(a, status, stream);
  const bool few = static_cast<int64_t>(a.rows) * (a.heads + 2 * a.kv_heads) < 64 * kNumSMs;
  return few ? launch_head_norm<T, 4, 1, 1>(a, status, stream) : launch_head_norm<T, 4, 1, 4>(a, status, stream);
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_head_norm_qkv(const B2HeadNormArgs* a, int f32, Status* status, cudaStream_t stream) {
  if (a->rows <= 0) return 0;
  if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->dim <= 0 || a->vdim <= 0 || a->v_off < 0 || a->pad_dim < a->dim ||
      a->pad_vdim < a->vdim || a->pad_dim > 256 || a->pad_vdim > 256 || a->page_size <= 0 || a->num_slots > 0x7fffffff || a->q_norm == nullptr || a->k_norm == nullptr)
    return -kBadArgument;
  return f32 ? dispatch_head_norm<float>(*a, status, stream) : dispatch_head_norm<__nv_bfloat16>(*a, status, stream);
}

extern "C" int b2_norm_qkv(const B2NormQkvArgs* a, int f32, Status* status, cudaStream_t stream) {
  if (a->rows <= 0) return 0;
  if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->dim <= 0 || a->vdim <= 0 || a->pad_dim < a->dim || a->pad_vdim < a->vdim ||
      a->rot < 0 || a->rot % 2 != 0 || a->rot > a->dim || a->page_size <= 0 || (a->rot > 0 && a->cos_sin == nullptr) ||
      static_cast<int64_t>(a->heads + a->kv_heads) * a->dim > 50000 || a->num_slots > 0x7fffffff)
    return -kBadArgument;
  // every vector access must be aligned: rows, heads, caches, and the table's two halves
  const bool v4 = a->dim % 4 == 0 && a->vdim % 4 == 0 && a->pad_dim % 4 == 0 && a->pad_vdim % 4 == 0 && a->ld % 4 == 0 && reinterpret_cast<uintptr_t>(a->proj) % 16 == 0;
  const bool v8 = a->dim >= 8 && a->dim <= 256 && (a->dim & (a->dim - 1)) == 0 && a->vdim == a->dim && a->rot % 16 == 0 && a->pad_dim % 8 == 0 &&
                  a->pad_vdim % 8 == 0 && a->ld % 8 == 0 && reinterpret_cast<uintptr_t>(a->proj) % 16 == 0;
  if (!f32 && v8 && a->rows >= 4 * kNumSMs && (a->heads + 2 * a->kv_heads) * a->dim <= 8192) return launch_norm_qkv_rows(*a, status, stream);
  if (v4 && a->dim <= 128 && a->vdim <= 128 && a->rot % 8 == 0 && a->heads + a->kv_heads <= 64)
    return f32 ? launch_norm_qkv_heads<float>(*a, status, stream) : launch_norm_qkv_heads<__nv_bfloat16>(*a, status, stream);
  if (f32) return v4 ? launch_norm_qkv<float, 4>(*a, status, stream) : launch_norm_qkv<float, 1>(*a, status, stream);
  return v4 ? launch_norm_qkv<__nv_bfloat16, 4>(*a, status, stream) : launch_norm_qkv<__nv_bfloat16, 1>(*a, status, stream);
}
