// Around latent attention: the normalised latent of every new token into its cache row (with the rotated key part that all heads
// share, while the queries rotate), and the latents of whole contexts out of their pages (for prompts, whose keys and values are then expanded by one matrix product).
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/latent.h"
#include "b2/launch.h"
#include "b2/ptx.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

// One warp: dst[0 : rank] = rms_norm(src) * weight, zeros up to `pad`. The row, up to 1024 columns, stays in registers.
template <typename T, int VEC>
__device__ __forceinline__ void write_latent(const T* src, const float* weight, float eps, T* dst, int rank, int pad, int lane) {
  constexpr int kMaxIt = 32 / VEC;
  float v[kMaxIt][VEC], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kMaxIt; ++i) {
    const int col = (i * 32 + lane) * VEC;
    if (col < rank) {
      load_f32<VEC>(src + col, v[i]);
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss = fmaf(v[i][j], v[i][j], ss);
    }
  }
  const float r = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(rank) + eps);
#pragma unroll
  for (int i = 0; i < kMaxIt; ++i) {
    const int col = (i * 32 + lane) * VEC;
    if (col >= pad) break;
    float w[VEC], o[VEC] = {};
    if (col < rank) {
      load_f32<VEC>(weight + col, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = v[i][j] * r * w[j];
    }
    store_f32<VEC>(dst + col, o);
  }
}

// One warp per token.
template <typename T, int VEC>
__global__ void __launch_bounds__(128) latent_write_kernel(const T* __restrict__ c, int64_t ld, const float* __restrict__ weight, float eps,
                                                           const int64_t* __restrict__ slots, T* __restrict__ cache, int rows, int rank, int pad,
                                                           int64_t num_slots, Status* status) {
  ptx::grid_dep_sync();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  const int64_t slot = slots[row];
  if (slot < 0 || !B2_ASSERT(status, slot < num_slots, kSiteKvIndex, slot, num_slots)) return;
  write_latent<T, VEC>(c + row * ld, weight, eps, cache + slot * pad, rank, pad, lane);
}

// One CTA per token: the first warp writes the cache row, all of them rotate the queries. PAIR: query pairs are aligned.
template <typename T, int VEC, bool PAIR>
__global__ void __launch_bounds__(128) latent_rope_kernel(const B2LatentRopeArgs a, Status* status) {
  ptx::grid_dep_sync();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = a.rot >> 1;
  int pos = a.positions[row];
  if (!B2_ASSERT(status, pos >= 0 && pos < a.max_pos, kSiteKvIndex, pos, a.max_pos)) pos = 0;
  const float* cs = a.cos_sin + static_cast<int64_t>(pos) * a.rot;
  const auto turn = [&](int i, float& u, float& v) {
    const float c = cs[i], s = cs[half + i], x = u;
    u = x * c - v * s;
    v = v * c + x * s;
  };
  if (warp == 0) {
    const int64_t slot = a.slots[row];
    if (slot >= 0 && B2_ASSERT(status, slot < a.num_slots, kSiteKvIndex, slot, a.num_slots)) {
      T* dst = static_cast<T*>(a.cache) + slot * a.pad;
      write_latent<T, VEC>(static_cast<const T*>(a.c) + row * a.ld, a.weight, a.eps, dst, a.rank, a.column, lane);
      const T* k = static_cast<const T*>(a.k) + row * a.ld;
      for (int i = lane; i < half; i += 32) {
        float u[1], v[1];
        load_f32<1>(k + 2 * i, u);
        load_f32<1>(k + 2 * i + 1, v);
        turn(i, u[0], v[0]);
        store_f32<1>(dst + a.column + 2 * i, u);
        store_f32<1>(dst + a.column + 2 * i + 1, v);
      }
      const float zero[1] = {0.0f};
      for (int i = a.column + a.rot + lane; i < a.pad; i += 32) store_f32<1>(dst + i, zero);
    }
  }
  T* q = static_cast<T*>(a.q) + row * a.ld_q + a.q_off;
  // the first warp has less of this to do
  for (int i = threadIdx.x < 32 ? a.heads * half : static_cast<int>(threadIdx.x) - 32; i < a.heads * half; i += 96) {
    const int h = i / half, p = i - h * half;
    T* at = q + static_cast<int64_t>(h) * a.q_dim + 2 * p;
    if constexpr (PAIR) {
      float uv[2];
      load_f32<2>(at, uv);
      turn(p, uv[0], uv[1]);
      store_f32<2>(at, uv);
    } else {
      float u[1], v[1];
      load_f32<1>(at, u);
      load_f32<1>(at + 1, v);
      turn(p, u[0], v[0]);
      store_f32<1>(at, u);
      store_f32<1>(at + 1, v);
    }
  }
}

template <typename T>
int launch_rope(const B2LatentRopeArgs& a, Status* status, cudaStream_t stream) {
  const uintptr_t addr = reinterpret_cast<uintptr_t>(a.c) | reinterpret_cast<uintptr_t>(a.cache);
  const bool v4 = a.rank % 4 == 0 && a.column % 4 == 0 && a.pad % 4 == 0 && a.ld % 4 == 0 && addr % 16 == 0;
  const bool pair = a.q_off % 2 == 0 && a.q_dim % 2 == 0 && a.ld_q % 2 == 0 && reinterpret_cast<uintptr_t>(a.q) % (2 * sizeof(T)) == 0;
  auto kern = v4 ? (pair ? latent_rope_kernel<T, 4, true> : latent_rope_kernel<T, 4, false>)
                 : (pair ? latent_rope_kernel<T, 1, true> : latent_rope_kernel<T, 1, false>);
  launch_pdl(kern, dim3(a.rows), dim3(128), 0, stream, a, status);
  return last_launch_rc();
}

template <typename T, int VEC>
int launch_write(const void* c, int64_t ld, const float* weight, float eps, const int64_t* slots, void* cache, int rows, int rank, int pad,
                 int64_t num_slots, Status* status, cudaStream_t stream) {
  if (pad > 1024) return -kTooLarge;
  launch_pdl(latent_write_kernel<T, VEC>, dim3((rows + 3) / 4), dim3(128), 0, stream, static_cast<const T*>(c), ld, weight, eps, slots,
             static_cast<T*>(cache), rows, rank, pad, num_slots, status);
  return last_launch_rc();
}

// One CTA per scratch page.
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* __restrict__ cache, const int32_t* __restrict__ pages,
                                                            const int32_t* __restrict__ ctx_lens, const int32_t* __restrict__ tables,
                                                            uint4* __restrict__ out, int seqs, int max_blocks, int page_size, int row_vecs,
                                                            int64_t num_pages, Status* status) {
  ptx::grid_dep_sync();
  const int seq = pages[2 * blockIdx.x], p0 = pages[2 * blockIdx.x + 1] * 128;
  const bool known = B2_ASSERT(status, seq >= 0 && seq < seqs && p0 >= 0, kSiteKvIndex, seq, p0);
  const int ctx = known ? ctx_lens[seq] : 0;
  uint4* dst = out + static_cast<int64_t>(blockIdx.x) * 128 * row_vecs;
  for (int i = threadIdx.x; i < 128 * row_vecs; i += blockDim.x) {
    const int r = i / row_vecs, v = i - r * row_vecs, pos = p0 + r;
    uint4 val = make_uint4(0, 0, 0, 0);
    if (pos < ctx) {
      const int block = pos / page_size;
      if (B2_ASSERT(status, block < max_blocks, kSiteKvIndex, block, max_blocks)) {
        const int64_t page = tables[static_cast<int64_t>(seq) * max_blocks + block];
        if (B2_ASSERT(status, page >= 0 && page < num_pages, kSiteKvIndex, page, num_pages))
          val = cache[(page * page_size + pos % page_size) * row_vecs + v];
      }
    }
    dst[i] = val;
  }
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_latent_write(const void* c, int64_t ld, const float* weight, float eps, const int64_t* slots, void* cache, int rows, int rank, int pad,
                               int64_t num_slots, int f32, Status* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (rank <= 0 || pad < rank) return -kBadArgument;
  const uintptr_t addr = reinterpret_cast<uintptr_t>(c) | reinterpret_cast<uintptr_t>(cache);
  const bool v4 = rank % 4 == 0 && pad % 4 == 0 && ld % 4 == 0 && addr % 16 == 0;
#define B2_WRITE(T, VEC) return launch_write<T, VEC>(c, ld, weight, eps, slots, cache, rows, rank, pad, num_slots, status, stream)
  if (f32) {
    if (v4) B2_WRITE(float, 4);
    B2_WRITE(float, 1);
  }
  if (v4) B2_WRITE(__nv_bfloat16, 4);
  B2_WRITE(__nv_bfloat16, 1);
#undef B2_WRITE
}

extern "C" int b2_latent_write_rope(const B2LatentRopeArgs* a, int f32, Status* status, cudaStream_t stream) {
  if (a->rows <= 0) return 0;
  if (a->rank <= 0 || a->rot <= 0 || a->rot % 2 != 0 || a->column < a->rank || a->column > 1024 || a->pad < a->column + a->rot || a->heads <= 0 ||
      a->q_off < 0 || a->q_off + a->rot > a->q_dim || a->ld_q < static_cast<int64_t>(a->heads) * a->q_dim)
    return -kBadArgument;
  return f32 ? launch_rope<float>(*a, status, stream) : launch_rope<__nv_bfloat16>(*a, status, stream);
}

extern "C" int b2_latent_gather_bf16(const void* cache, const int32_t* pages, const int32_t* ctx_lens, const int32_t* block_tables, void* out,
                                     int n_pages, int seqs, int max_blocks, int page_size, int pad, int64_t num_pages, Status* status,
                                     cudaStream_t stream) {
  if (n_pages <= 0) return 0;
  if (pad % 8 != 0 || page_size <= 0) return -kBadArgument;
  launch_pdl(latent_gather_kernel, dim3(n_pages), dim3(256), 0, stream, static_cast<const uint4*>(cache), pages, ctx_lens, block_tables,
             static_cast<uint4*>(out), seqs, max_blocks, page_size, pad / 8, num_pages, status);
  return last_launch_rc();
}
