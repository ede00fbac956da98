// Epilogue of the grouped expert products: weights are the 128-row UMMA M side, the tokens of one expert the N side.
// A unit's q_coord is its first row in the token matrix (input and output rows coincide), nsplit the number of its rows
// that hold tokens.
#pragma once
#include <cuda_bf16.h>
#include "b2/act.cuh"
#include "b2/gemm_tc.cuh"
#include "b2/ptx.cuh"

namespace b2 {

struct GroupedEpiParams {
  __nv_bfloat16* y;
  int64_t ldy;
  int n_rows;      // rows of one expert's weight
  int mode;        // B2_EPI_NONE, B2_EPI_RELU2 or B2_EPI_SWIGLU
  B2EpiAct act;
};

template <int BN>
struct GroupedEpilogue {
  static constexpr int CH = BN >= 32 ? 32 : 16;
  GroupedEpiParams p;
  __device__ __forceinline__ void operator()(const gemm::WorkUnit& u, uint32_t taddr, int quarter, int lane, uint32_t*,
                                             Status*) const {
    const int p_local = quarter * 32 + lane;
    const int n = u.pb * 128 + p_local;
    __nv_bfloat16* base = p.y + static_cast<int64_t>(u.q_coord) * p.ldy;
#pragma unroll 1
    for (int c = 0; c < BN / CH; ++c) {
      const int m0 = c * CH;
      if (m0 >= u.nsplit) break;
      uint32_t r[CH];
      if constexpr (CH == 32) ptx::tmem_ld_32x32(taddr + c * CH, r);
      else ptx::tmem_ld_32x16(taddr + c * CH, r);
      ptx::tc_wait_ld();
      if (p.mode == B2_EPI_SWIGLU) {
        const int out_col = (u.pb * 128 + (p_local & ~31)) / 2 + (lane & 15);
#pragma unroll
        for (int j = 0; j < CH; ++j) {
          const float v = __uint_as_float(r[j]);
          const float other = __shfl_xor_sync(0xffffffffu, v, 16);
          if (lane < 16 && n < p.n_rows && m0 + j < u.nsplit)
            base[static_cast<int64_t>(m0 + j) * p.ldy + out_col] = __float2bfloat16(glu(p.act, v, other));
        }
      } else if (n < p.n_rows) {
#pragma unroll
        for (int j = 0; j < CH; ++j) {
          if (m0 + j >= u.nsplit) break;
          const float v = __uint_as_float(r[j]);
          base[static_cast<int64_t>(m0 + j) * p.ldy + n] = __float2bfloat16(p.mode == B2_EPI_RELU2 ? relu2(v) : v);
        }
      }
    }
  }
};

constexpr int grouped_stages_for(int bn) {
  const int stage = 128 * 64 * 2 + bn * 64 * 2;
  const int s = (200 * 1024) / stage;
  return s > 10 ? 10 : s;
}

}  // namespace b2
