// Mixture-of-experts layers whose experts all live on this GPU: routing, the permutation of the token rows, and the grouped
// expert products over a packed list of tiles. No counts travel to the host, so a layer can sit in a CUDA graph; memory is
// rows * top, whatever the split over the experts. The weighted sum of the results is part of the residual kernel
// (residual_norm.cu).
#include <cstdint>
#include <cuda.h>
#include <cuda_bf16.h>
#include "b2/elem.cuh"
#include "b2/latent.h"
#include "b2/launch.h"
#include "b2/moe_gemm.cuh"
#include "b2/ptx.cuh"
#include "b2/tma.h"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kMaxTop = 32;
constexpr int kMaxExperts = 1024;

// Index of the largest value over a warp's NV * 32 (lane + 32 i), lowest index on ties; `none` where nothing compares.
template <int NV>
__device__ __forceinline__ int warp_argmax(const float (&v)[NV], int lane, int none, float& best) {
  best = -INFINITY;
  int at = none;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (v[i] > best) { best = v[i]; at = lane + 32 * i; }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ob = __shfl_xor_sync(0xffffffffu, best, o);
    const int oe = __shfl_xor_sync(0xffffffffu, at, o);
    if (ob > best || (ob == best && oe < at)) { best = ob; at = oe; }
  }
  return min(at, none);
}

// One warp per row, NV logits per lane. The largest logits have the largest scores, and differ where scores are as good as one.
// CHOICE: what chooses is not the score itself (a correction is added, groups are left out); then scores and choice scores are held
// apart.
template <int NV, bool CHOICE>
__global__ void __launch_bounds__(256) moe_route_kernel(const float* __restrict__ logits, int64_t ld, const float* __restrict__ correction,
                                                        float* __restrict__ weights, int32_t* __restrict__ ids, int32_t* __restrict__ place,
                                                        int32_t* __restrict__ counts, int rows, int experts, int outputs, int top, int groups, int keep,
                                                        int sigmoid, int norm_top, float scale) {
  ptx::grid_dep_sync();
  __shared__ float pool[CHOICE ? 8 : 1][CHOICE ? NV * 32 : 1];
  const int row = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (row >= rows) return;
  float v[NV], mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = lane + 32 * i;
    v[i] = e < outputs ? logits[row * ld + e] : -INFINITY;
    mx = fmaxf(mx, v[i]);
  }
  float inv = 1.0f;
  const auto score_of = [&](float logit) { return sigmoid ? sigmoid_f32(logit) : expf(logit - mx); };
  if (!sigmoid) mx = warp_max(mx);
  if (CHOICE || !sigmoid) {
    float sum = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const float p = lane + 32 * i < outputs ? score_of(v[i]) : -INFINITY;
      if (p > 0.0f) sum += p;
      if constexpr (CHOICE) v[i] = p;
    }
    if (!sigmoid) inv = 1.0f / warp_sum(sum);
  }
  float score[CHOICE ? NV : 1];
  if constexpr (CHOICE) {
    float* mine = pool[threadIdx.x >> 5];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = lane + 32 * i;
      score[i] = v[i] * inv;
      v[i] = e < outputs ? score[i] + (correction != nullptr ? correction[e] : 0.0f) : -INFINITY;
      mine[e] = v[i];
    }
    inv = 1.0f;
    if (keep < groups) {
      const int per = outputs / groups;
      float gm[NV];
      uint32_t kept = 0;
      __syncwarp();
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        gm[i] = -INFINITY;
        if (lane + 32 * i < groups)
          for (int j = 0; j < per; ++j) gm[i] = fmaxf(gm[i], mine[(lane + 32 * i) * per + j]);
      }
      for (int j = 0; j < keep; ++j) {
        float best;
        const int g = warp_argmax<NV>(gm, lane, groups - 1, best);
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (g == lane + 32 * i) {
            gm[i] = -INFINITY;
            kept |= 1u << i;
          }
      }
      __syncwarp();
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (lane + 32 * i < groups) mine[lane + 32 * i] = (kept >> i) & 1u ? 1.0f : 0.0f;
      __syncwarp();
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (lane + 32 * i < outputs && mine[(lane + 32 * i) / per] == 0.0f) v[i] = -INFINITY;
    }
  }
  float sel_w = 0.0f, total = 0.0f;   // lane j keeps the j-th choice
  int sel_e = 0;
  for (int j = 0; j < top; ++j) {
    float best;
    const int best_e = warp_argmax<NV>(v, lane, outputs - 1, best);    // where nothing compares (NaN logits): still a valid output
    if constexpr (CHOICE) {
      float own = 0.0f;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (best_e == lane + 32 * i) own = score[i];
      best = __shfl_sync(0xffffffffu, own, best_e & 31);
    } else {
      best = score_of(best);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (best_e == lane + 32 * i) v[i] = -INFINITY;   // out of the pool
    if (lane == j) { sel_w = best * inv; sel_e = best_e; }
    total += best * inv;
  }
  if (lane < top) {
    if (norm_top) sel_w /= total + 1e-20f;
    const int64_t at = static_cast<int64_t>(row) * top + lane;
    weights[at] = sel_w * scale;
    ids[at] = sel_e;
    place[at] = sel_e < experts ? atomicAdd(counts + sel_e, 1) : 0;
  }
}

// 16 bytes of a row times f.
template <typename T>
__device__ __forceinline__ uint4 scaled(uint4 r, float f) {
  if constexpr (sizeof(T) == 4) {
    return make_uint4(__float_as_uint(__uint_as_float(r.x) * f), __float_as_uint(__uint_as_float(r.y) * f), __float_as_uint(__uint_as_float(r.z) * f),
                      __float_as_uint(__uint_as_float(r.w) * f));
  } else {
    float v[8];
    bf16x8_to_f32(r, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= f;
    return f32_to_bf16x8(v);
  }
}

// Every CTA forms the experts' first rows itself (a scan over the counts); CTA 0 also lists the tiles. Then one warp per
// row copies it to its `top` places, times the choice's weight where `weights` are given. The order inside an expert is the order of the atomics above and does not touch any
// result: a row's product depends on that row alone.
template <typename T>
__global__ void __launch_bounds__(256) moe_gather_kernel(const T* __restrict__ x, const int32_t* __restrict__ ids, const int32_t* __restrict__ place,
                                                         const float* __restrict__ weights,
                                                         int32_t* __restrict__ counts, int32_t* __restrict__ slot, T* __restrict__ xs,
                                                         int4* __restrict__ tiles, int32_t* __restrict__ n_tiles, int rows, int experts, int top,
                                                         int width, int bn, int max_tiles, Status* status) {
  ptx::grid_dep_sync();
  __shared__ int first[kMaxExperts];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) {
    int row0 = 0, tile0 = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      const int e = e0 + lane, cnt = e < experts ? __ldcg(counts + e) : 0, nt = (cnt + bn - 1) / bn;
      int rs = cnt, ts = nt;      // inclusive scans over the warp
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, rs, o), b = __shfl_up_sync(0xffffffffu, ts, o);
        if (lane >= o) { rs += a; ts += b; }
      }
      if (e < experts) first[e] = row0 + rs - cnt;
      if (blockIdx.x == 0)
        for (int t = 0; t < nt; ++t) {
          const int at = tile0 + ts - nt + t;
          if (B2_ASSERT(status, at < max_tiles, kSiteEpCount, at, max_tiles)) tiles[at] = make_int4(e, row0 + rs - cnt + t * bn, min(bn, cnt - t * bn), 0);
        }
      row0 += __shfl_sync(0xffffffffu, rs, 31);
      tile0 += __shfl_sync(0xffffffffu, ts, 31);
    }
    if (blockIdx.x == 0 && lane == 0) n_tiles[0] = min(tile0, max_tiles);
  }
  __syncthreads();
  // the CTA that is last to have read the counts leaves them at zero for the next layer
  __shared__ int last;
  if (threadIdx.x == 0) last = atomicAdd(counts + experts, 1) == static_cast<int>(gridDim.x) - 1;
  __syncthreads();
  if (last)
    for (int e = threadIdx.x; e <= experts; e += blockDim.x) counts[e] = 0;
  const int vecs = width * static_cast<int>(sizeof(T)) / 16, n_warps = gridDim.x * 8;
  for (int t = blockIdx.x * 8 + warp; t < rows; t += n_warps) {
    int mine = 0;
    float mine_w = 1.0f;
    if (lane < top) {
      const int64_t at = static_cast<int64_t>(t) * top + lane;
      if (weights != nullptr) mine_w = weights[at];
      const int id = ids[at];
      mine = id < experts ? first[id] + place[at] : -1;      // what returns its input needs no copy of it
      if (!B2_ASSERT(status, mine >= -1 && mine < rows * top, kSiteEpCount, mine, rows * top)) mine = 0;
      slot[at] = mine;
    }
    const uint4* src = reinterpret_cast<const uint4*>(x) + static_cast<int64_t>(t) * vecs;
    for (int c0 = 0; c0 < vecs; c0 += 128) {     // warp-uniform trip count
      uint4 r[4];
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (c0 + u * 32 + lane < vecs) r[u] = ptx::ld_nc_v4(src + c0 + u * 32 + lane);
      for (int j = 0; j < top; ++j) {
        const int to = __shfl_sync(0xffffffffu, mine, j);
        const float f = __shfl_sync(0xffffffffu, mine_w, j);
        if (to < 0) continue;
        uint4* dst = reinterpret_cast<uint4*>(xs) + static_cast<int64_t>(to) * vecs;
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (c0 + u * 32 + lane < vecs) dst[c0 + u * 32 + lane] = weights != nullptr ? scaled<T>(r[u], f) : r[u];
      }
    }
  }
}

// Units (tile, 128 weight rows) over the device-side tile list; consecutive units share the token tile.
struct TileListSched {
  const int4* tiles;
  const int32_t* n_tiles;
  int n_rows, num_kb, p_blocks;
  __device__ __forceinline__ int total() const { return *n_tiles * p_blocks; }
  __device__ __forceinline__ gemm::WorkUnit get(int w) const {
    gemm::WorkUnit u;
    u.qb = w / p_blocks;
    u.pb = w - u.qb * p_blocks;
    const int4 t = tiles[u.qb];
    u.split = t.x;
    u.tile = w;
    u.kb0 = 0;
    u.kb1 = num_kb;
    u.nsplit = t.z;
    u.p_coord = t.x * n_rows + u.pb * gemm::kBlockP;
    u.q_coord = t.y;
    return u;
  }
};

template <int BN, int STAGES>
__global__ void __launch_bounds__(gemm::kThreads, 1)
moe_tiles_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x, TileListSched sched, GroupedEpiParams ep,
                 Status* status) {
  constexpr uint32_t idesc = ptx::make_idesc(1, 1, 128, BN);
  GroupedEpilogue<BN> epi{ep};
  gemm::run<BN, STAGES, 2>(&tmap_w, &tmap_x, idesc, ptx::kEvictFirst, ptx::kEvictLast, sched, gemm::NoGate{}, epi, status,
                           static_cast<int>(blockIdx.x), static_cast<int>(gridDim.x));
}

template <int BN>
int launch_tiles(const void* x, const void* w, const int32_t* tiles, const int32_t* n_tiles, void* y, int rows, int experts, int n, int k, int epilogue,
                 const B2EpiAct* act, Status* status, cudaStream_t stream) {
  constexpr int STAGES = grouped_stages_for(BN);
  using L = gemm::SmemLayout<BN, STAGES>;
  CUtensorMap tw, tx;
  if (!make_tmap_2d(&tw, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, w, static_cast<uint64_t>(experts) * n, k, static_cast<uint64_t>(k) * 2, 128, 64,
                    CU_TENSOR_MAP_SWIZZLE_128B) ||
      !make_tmap_2d(&tx, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, x, rows, k, static_cast<uint64_t>(k) * 2, BN, 64, CU_TENSOR_MAP_SWIZZLE_128B))
    return -kBadArgument;
  const TileListSched sched{reinterpret_cast<const int4*>(tiles), n_tiles, n, (k + 63) / 64, (n + 127) / 128};
  const GroupedEpiParams ep{static_cast<__nv_bfloat16*>(y), epilogue == B2_EPI_SWIGLU ? n / 2 : n, n, epilogue, act != nullptr ? *act : kPlainAct};
  auto kern = moe_tiles_kernel<BN, STAGES>;
  static DeviceOnce attr_once;
  if (const int rc = attr_once.max_smem(kern, L::kTotalBytes)) return rc;
  launch_pdl(kern, dim3(kNumSMs), dim3(gemm::kThreads), L::kTotalBytes, stream, tw, tx, sched, ep, status);
  return last_launch_rc();
}

// 64 x 64 tile, 256 threads of 4 x 4 outputs.
__global__ void __launch_bounds__(256) moe_tiles_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, const int4* __restrict__ tiles,
                                                            const int32_t* __restrict__ n_tiles, float* __restrict__ y, int n, int k, int epilogue) {
  ptx::grid_dep_sync();
  if (static_cast<int>(blockIdx.y) >= *n_tiles) return;
  const int4 tile = tiles[blockIdx.y];
  __shared__ float xs[16][68], ws[16][68];
  const float* xr = x + static_cast<int64_t>(tile.y) * k;
  const float* wr = w + static_cast<int64_t>(tile.x) * n * k;
  const int n0 = blockIdx.x * 64, tm = (threadIdx.x >> 4) * 4, tn = (threadIdx.x & 15) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i / 16, c = i % 16;
      xs[c][r] = r < tile.z && k0 + c < k ? xr[static_cast<int64_t>(r) * k + k0 + c] : 0.0f;
      ws[c][r] = n0 + r < n && k0 + c < k ? wr[static_cast<int64_t>(n0 + r) * k + k0 + c] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 16; ++c) {
      float a[4], b[4];
      load_f32<4>(&xs[c][tm], a);
      load_f32<4>(&ws[c][tn], b);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (tm + i < tile.z && n0 + tn + j < n) y[static_cast<int64_t>(tile.y + tm + i) * n + n0 + tn + j] = epilogue == B2_EPI_RELU2 ? relu2(acc[i][j]) : acc[i][j];
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_moe_route(const float* logits, int64_t ld, const float* correction, float* weights, int32_t* ids, int32_t* place, int32_t* counts,
                            int rows, int experts, int identity, int top, int groups, int keep, int scoring, int norm_top, float scale,
                            cudaStream_t stream) {
  if (rows <= 0) return 0;
  const int outputs = experts + identity;
  if (experts < 1 || identity < 0 || outputs > kMaxExperts || groups < 1 || outputs % groups != 0 || keep < 1 || keep > groups || top < 1 || top > kMaxTop ||
      top > outputs / groups * keep || ld < outputs || scoring < 0 || scoring > 1)
    return -kBadArgument;
  const bool choice = correction != nullptr || keep < groups;
  auto kern = outputs <= 256 ? (choice ? moe_route_kernel<8, true> : moe_route_kernel<8, false>)
                             : (choice ? moe_route_kernel<32, true> : moe_route_kernel<32, false>);
  launch_pdl(kern, dim3((rows + 7) / 8), dim3(256), 0, stream, logits, ld, correction, weights, ids, place, counts, rows, experts, outputs, top, groups, keep,
             scoring, norm_top, scale);
  return last_launch_rc();
}

extern "C" int b2_moe_gather(const void* x, const int32_t* ids, const int32_t* place, const float* weights, int32_t* counts, int32_t* slot, void* xs, int32_t* tiles,
                             int32_t* n_tiles, int rows, int experts, int top, int width, int bn, int f32, Status* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  const int esz = f32 ? 4 : 2;
  if (experts < 1 || experts > kMaxExperts || top < 1 || top > kMaxTop || bn < 1 || width <= 0 || width * esz % 16 != 0 ||
      static_cast<int64_t>(rows) * top > (1 << 30) || (reinterpret_cast<uintptr_t>(x) & 15) != 0 || (reinterpret_cast<uintptr_t>(xs) & 15) != 0)
    return -kBadArgument;
  const int blocks = (rows + 7) / 8 < 2 * kNumSMs ? (rows + 7) / 8 : 2 * kNumSMs, max_tiles = experts + rows * top / bn;
  if (f32)
    launch_pdl(moe_gather_kernel<float>, dim3(blocks), dim3(256), 0, stream, static_cast<const float*>(x), ids, place, weights, counts, slot, static_cast<float*>(xs),
               reinterpret_cast<int4*>(tiles), n_tiles, rows, experts, top, width, bn, max_tiles, status);
  else
    launch_pdl(moe_gather_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, static_cast<const __nv_bfloat16*>(x), ids, place, weights, counts, slot,
               static_cast<__nv_bfloat16*>(xs), reinterpret_cast<int4*>(tiles), n_tiles, rows, experts, top, width, bn, max_tiles, status);
  return last_launch_rc();
}

extern "C" int b2_moe_tiles_gemm_bf16(const void* x, const void* w, const int32_t* tiles, const int32_t* n_tiles, void* y, int rows, int experts, int n,
                                      int k, int epilogue, const B2EpiAct* act, int bn, Status* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (experts < 1 || n <= 0 || k <= 0 || k % 8 != 0 || (epilogue != B2_EPI_NONE && epilogue != B2_EPI_RELU2 && epilogue != B2_EPI_SWIGLU) || (epilogue == B2_EPI_SWIGLU && n % 32 != 0))
    return -kBadArgument;
  switch (bn) {
    case 16: return launch_tiles<16>(x, w, tiles, n_tiles, y, rows, experts, n, k, epilogue, act, status, stream);
    case 32: return launch_tiles<32>(x, w, tiles, n_tiles, y, rows, experts, n, k, epilogue, act, status, stream);
    case 64: return launch_tiles<64>(x, w, tiles, n_tiles, y, rows, experts, n, k, epilogue, act, status, stream);
    case 128: return launch_tiles<128>(x, w, tiles, n_tiles, y, rows, experts, n, k, epilogue, act, status, stream);
    case 256: return launch_tiles<256>(x, w, tiles, n_tiles, y, rows, experts, n, k, epilogue, act, status, stream);
    default: return -kBadArgument;
  }
}

extern "C" int b2_moe_tiles_gemm_f32(const float* x, const float* w, const int32_t* tiles, const int32_t* n_tiles, float* y, int max_tiles, int n, int k,
                                     int epilogue, cudaStream_t stream) {
  if (max_tiles <= 0) return 0;
  if (n <= 0 || k <= 0 || max_tiles > 65535 || (epilogue != B2_EPI_NONE && epilogue != B2_EPI_RELU2)) return -kBadArgument;
  launch_pdl(moe_tiles_f32_kernel, dim3((n + 63) / 64, max_tiles), dim3(256), 0, stream, x, w, reinterpret_cast<const int4*>(tiles), n_tiles, y, n, k, epilogue);
  return last_launch_rc();
}
