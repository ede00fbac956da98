// One small matrix per head: y[t, h, :] = W_h x[t, h, :] for the heads of a row laid side by side, on the tcgen05 core.
// The token rows are the P operand, read at the head's columns; a head's weight rows are the Q operand. Optional output
// gate: every element is multiplied by the sigmoid of its own logit, or of its head's, before it is rounded.
#include <cstdint>
#include <cuda.h>
#include <cuda_bf16.h>
#include "b2/gemm_tc.cuh"
#include "b2/latent.h"
#include "b2/launch.h"
#include "b2/ptx.cuh"
#include "b2/tma.h"
#include "b2/vec.cuh"

namespace b2 {
namespace {

struct HeadSched {
  int row_tiles, n_tiles, heads, n, k_dim, bn;
  __device__ __forceinline__ int total() const { return row_tiles * n_tiles * heads; }
  __device__ __forceinline__ gemm::WorkUnit get(int w) const {
    gemm::WorkUnit u;
    const int per_head = row_tiles * n_tiles;
    u.split = w / per_head;                   // carries the head
    const int r = w - u.split * per_head;
    u.pb = r % row_tiles;                     // consecutive units share the weight tile
    u.qb = r / row_tiles;
    u.kb0 = 0;
    u.kb1 = k_dim / gemm::kBlockK;
    u.tile = w;
    u.nsplit = 1;
    u.p_coord = u.pb * gemm::kBlockP;
    u.q_coord = u.split * n + u.qb * bn;
    return u;
  }
  __device__ __forceinline__ int p_kx(const gemm::WorkUnit& u) const { return u.split * k_dim; }
};

template <int BN>
struct HeadEpilogue {
  __nv_bfloat16* y;
  const __nv_bfloat16* gate;
  int64_t ldy, ld_gate;
  int rows, n, gate_heads;
  __device__ __forceinline__ void operator()(const gemm::WorkUnit& u, uint32_t taddr, int quarter, int lane, uint32_t*, Status*) const {
    const int row = u.pb * gemm::kBlockP + quarter * 32 + lane;
    const int64_t col0 = static_cast<int64_t>(u.split) * n + u.qb * BN;
    const bool by_head = gate != nullptr && gate_heads;
    float f_head = 1.0f;
    if (by_head && row < rows) f_head = ptx::rcp(1.0f + ptx::ex2(-__bfloat162float(gate[row * ld_gate + u.split]) * ptx::kLog2e));
#pragma unroll 1
    for (int c = 0; c < BN / 32; ++c) {
      uint32_t r[32];
      ptx::tmem_ld_32x32(taddr + c * 32, r);
      ptx::tc_wait_ld();
      if (row >= rows) continue;
      __nv_bfloat16* dst = y + row * ldy + col0 + c * 32;
      const __nv_bfloat16* z = gate != nullptr && !by_head ? gate + row * ld_gate + col0 + c * 32 : nullptr;
#pragma unroll
      for (int g = 0; g < 4; ++g) {
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(r[g * 8 + i]) * f_head;
        if (z != nullptr) {
          float f[8];
          bf16x8_to_f32(ptx::ld_v4(z + g * 8), f);
#pragma unroll
          for (int i = 0; i < 8; ++i) v[i] *= ptx::rcp(1.0f + ptx::ex2(-f[i] * ptx::kLog2e));
        }
        ptx::st_v4(dst + g * 8, f32_to_bf16x8(v));
      }
    }
  }
};

template <int BN, int STAGES>
__global__ void __launch_bounds__(gemm::kThreads, 1)
head_gemm_kernel(const __grid_constant__ CUtensorMap tmap_x, const __grid_constant__ CUtensorMap tmap_w, HeadSched sched, HeadEpilogue<BN> epi,
                 Status* status) {
  constexpr uint32_t idesc = ptx::make_idesc(1, 1, 128, BN);
  gemm::run<BN, STAGES, 2>(&tmap_x, &tmap_w, idesc, ptx::kEvictNormal, ptx::kEvictLast, sched, gemm::NoGate{}, epi, status,
                           static_cast<int>(blockIdx.x), static_cast<int>(gridDim.x));
}

template <int BN>
int launch_head(const void* x, const void* w, void* y, const void* gate, int rows, int heads, int n, int k_dim, int64_t ldx, int64_t ldw, int64_t ldy, int64_t ld_gate,
                int gate_heads, Status* status, cudaStream_t stream) {
  constexpr int STAGES = 6;
  using L = gemm::SmemLayout<BN, STAGES>;
  CUtensorMap tx, tw;
  if (!make_tmap_2d(&tx, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, x, rows, static_cast<uint64_t>(heads) * k_dim, ldx * 2, 128, 64, CU_TENSOR_MAP_SWIZZLE_128B) ||
      !make_tmap_2d(&tw, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, w, static_cast<uint64_t>(heads) * n, k_dim, ldw * 2, BN, 64,
                    CU_TENSOR_MAP_SWIZZLE_128B))
    return -kBadArgument;
  const HeadSched sched{(rows + 127) / 128, n / BN, heads, n, k_dim, BN};
  const HeadEpilogue<BN> epi{static_cast<__nv_bfloat16*>(y), static_cast<const __nv_bfloat16*>(gate), ldy, ld_gate, rows, n, gate_heads};
  auto kern = head_gemm_kernel<BN, STAGES>;
  static DeviceOnce attr_once;
  if (const int rc = attr_once.max_smem(kern, L::kTotalBytes)) return rc;
  const int64_t units = static_cast<int64_t>(sched.row_tiles) * sched.n_tiles * heads;
  launch_pdl(kern, dim3(units < kNumSMs ? static_cast<int>(units) : kNumSMs), dim3(gemm::kThreads), L::kTotalBytes, stream, tx, tw, sched, epi, status);
  return last_launch_rc();
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_head_gemm_bf16(const void* x, const void* w, void* y, const void* gate, int rows, int heads, int n, int k_dim, int64_t ldx, int64_t ldw,
                                 int64_t ldy, int64_t ld_gate, int gate_heads, Status* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (heads <= 0 || n <= 0 || n % 64 != 0 || k_dim <= 0 || k_dim % 64 != 0 || ldx % 8 != 0 || ldw % 8 != 0 || ldw < k_dim || ldy % 8 != 0 || (reinterpret_cast<uintptr_t>(y) & 15) != 0 ||
      (gate != nullptr && !gate_heads && (ld_gate % 8 != 0 || (reinterpret_cast<uintptr_t>(gate) & 15) != 0)))
    return -kBadArgument;
  // wide tiles once they alone fill the machine
  const int64_t wide = static_cast<int64_t>((rows + 127) / 128) * heads * (n / 128);
  if (n % 128 == 0 && wide >= kNumSMs) return launch_head<128>(x, w, y, gate, rows, heads, n, k_dim, ldx, ldw, ldy, ld_gate, gate_heads, status, stream);
  return launch_head<64>(x, w, y, gate, rows, heads, n, k_dim, ldx, ldw, ldy, ld_gate, gate_heads, status, stream);
}
