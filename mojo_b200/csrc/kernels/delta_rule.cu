// Gated delta rule with one decay per key channel. State S [dim, vdim] per head, all of it in f32:
//   S <- g * S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q
// Three kernels:
//   prep    every row and head at once: short convolution and silu of q, k, v, unit norms, decays, step sizes, and the few
//           dot products of neighbouring rows that the scan needs; f32, laid out the way the other two read them
//   decode  one row per sequence. CTA = (head, sequence): S streams through registers once, output norm and gate fused
//   scan    any number of rows. CTA = (32 value columns, head, sequence): S stays in the registers of four warps, which walk
//           over the rows two at a time while bulk copies bring the next rows into shared memory; norm and gate follow in a
//           kernel of their own
// S^T k and S^T q are read off the decayed state together, and the new write's share u (k . q) is added to the output, so a
// row costs one pass over S. Two rows at a time: with A = g1 * S, the second row reads g2 * A, to which the first row's write
// contributes u1 ((g2 k1) . k2) and u1 ((g2 k1) . q2); both rows' sums come out of one reduction.
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/short_conv.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kMaxDim = 256;
constexpr float kUnitEps = 1e-6f;
constexpr int kTile = 16;        // rows of one shared-memory stage of the scan
constexpr int kStages = 3;
constexpr int kCols = 32;        // value columns of a scan CTA

__device__ __forceinline__ float silu_f32(float x) { return x / (1.0f + expf(-x)); }

// Prepared rows, f32, head-major so that a tile of rows is one contiguous block:
//   qkg [heads][rows][3][kd]            unit q (times dim^-0.5), unit k, decay; zero / zero / one past dim
//   v   [heads][col blocks][rows][32]
//   sc  [heads][rows][4]                beta, k . q, and for every second row of a sequence (g k') . k and (g k') . q, where k'
//                                       is the row before
struct Prepared {
  float* qkg;
  float* v;
  float* sc;
  int kd, blocks, rows;
  __device__ __forceinline__ float* qkg_row(int h, int row) const { return qkg + (static_cast<int64_t>(h) * rows + row) * 3 * kd; }
  __device__ __forceinline__ float* v_row(int h, int blk, int row) const { return v + ((static_cast<int64_t>(h) * blocks + blk) * rows + row) * kCols; }
  __device__ __forceinline__ float* sc_row(int h, int row) const { return sc + (static_cast<int64_t>(h) * rows + row) * 4; }
};

int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
int64_t scratch_floats(int heads, int dim, int vdim, int rows) {
  const int64_t blocks = (vdim + kCols - 1) / kCols;
  return static_cast<int64_t>(rows) * heads * (3 * padded_dim(dim) + blocks * kCols + 4);
}
Prepared prepared_of(const B2DeltaArgs& a, int rows) {
  Prepared p;
  p.kd = padded_dim(a.dim);
  p.blocks = (a.vdim + kCols - 1) / kCols;
  p.rows = rows;
  p.qkg = a.scratch;
  p.v = p.qkg + static_cast<int64_t>(rows) * a.heads * 3 * p.kd;
  p.sc = p.v + static_cast<int64_t>(rows) * a.heads * p.blocks * kCols;
  return p;
}

// ------------------------------------------------------------------------------------------------------------
// prep
// ------------------------------------------------------------------------------------------------------------
// Warp = (TT consecutive rows of one sequence, head); tiles count from each sequence's first row, so a pair of rows never
// straddles two warps. Lane l holds channels (l + 32 j) * VEC.
template <typename T, int VEC, int NJ, int TAPS, int TT>
__global__ void __launch_bounds__(128) delta_prep_kernel(const B2DeltaArgs a, const B2SeqRows sq, const Prepared out, Status* status) {
  ptx::grid_dep_sync();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * 4 + warp;
  if (h >= a.heads) return;
  // which sequence tile number blockIdx.x belongs to: 32 sequences at a time, prefix sum over the lanes
  int seq = -1, tile = static_cast<int>(blockIdx.x);
  for (int s0 = 0; s0 < sq.seqs && seq < 0; s0 += 32) {
    int tiles = 0;
    if (s0 + lane < sq.seqs) tiles = (max(0, sq.seq_rows[2 * (s0 + lane) + 1] - sq.seq_rows[2 * (s0 + lane)]) + TT - 1) / TT;
    int sum = tiles;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += up;
    }
    const uint32_t hit = __ballot_sync(0xffffffffu, tile < sum);
    if (hit != 0) {
      const int l = __ffs(hit) - 1;
      seq = s0 + l;
      tile -= __shfl_sync(0xffffffffu, sum - tiles, l);
    } else {
      tile -= __shfl_sync(0xffffffffu, sum, 31);
    }
  }
  if (seq < 0) return;
  const int row0 = sq.seq_rows[2 * seq] + tile * TT;
  ConvRow cr;
  if (!cr.load(sq, seq, row0, sq.banks, status)) return;
  const int n = min(TT, cr.end - row0);
  const int d = a.dim, e = a.vdim, per = a.heads / a.kv_heads, kh = h / per, ck = a.kv_heads * d;
  const ConvSource<T> src{static_cast<const T*>(a.proj), a.ld, a.conv_w, static_cast<T*>(a.conv_state), a.taps, 2 * ck + a.heads * e, sq.banks};
  const bool save_qk = h % per == 0;

  float q[NJ][TT][VEC], k[NJ][TT][VEC], g[NJ][TT][VEC];
  const float neg_rate = a.neg_rate[h];
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
    if (c < d) {
      conv_rows<T, VEC, TAPS, TT>(src, cr, row0, n, kh * d + c, save_qk, q[j]);
      conv_rows<T, VEC, TAPS, TT>(src, cr, row0, n, ck + kh * d + c, save_qk, k[j]);
      float bias[VEC];
      load_f32<VEC>(a.dt_bias + h * d + c, bias);
#pragma unroll
      for (int t = 0; t < TT; ++t) {
        float z[VEC] = {};
        if (t < n) load_f32<VEC>(static_cast<const T*>(a.dg) + static_cast<int64_t>(row0 + t) * a.ld_dg + h * d + c, z);
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          q[j][t][v] = silu_f32(q[j][t][v]);
          k[j][t][v] = silu_f32(k[j][t][v]);
          g[j][t][v] = expf(neg_rate * softplus_f32(z[v] + bias[v]));
        }
      }
    } else {
#pragma unroll
      for (int t = 0; t < TT; ++t)
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          q[j][t][v] = k[j][t][v] = 0.0f;
          g[j][t][v] = 1.0f;
        }
    }
  }
  const float q_scale = rsqrtf(static_cast<float>(d));
#pragma unroll
  for (int t = 0; t < TT; ++t) {
    if (t >= n) break;
    float qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        qq = fmaf(q[j][t][v], q[j][t][v], qq);
        kk = fmaf(k[j][t][v], k[j][t][v], kk);
        qk = fmaf(q[j][t][v], k[j][t][v], qk);
      }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    qk = warp_sum(qk);
    const float rq = q_scale / sqrtf(qq + kUnitEps), rk = 1.0f / sqrtf(kk + kUnitEps);
    float* dst = out.qkg_row(h, row0 + t);
    float gkk = 0.0f, gkq = 0.0f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = (lane + 32 * j) * VEC;
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        q[j][t][v] *= rq;
        k[j][t][v] *= rk;
        if (t & 1) {
          const float gk = g[j][t][v] * k[j][t - (t & 1)][v];
          gkk = fmaf(gk, k[j][t][v], gkk);
          gkq = fmaf(gk, q[j][t][v], gkq);
        }
      }
      if (c < out.kd) {
        store_f32<VEC>(dst + c, q[j][t]);
        store_f32<VEC>(dst + out.kd + c, k[j][t]);
        store_f32<VEC>(dst + 2 * out.kd + c, g[j][t]);
      }
    }
    if (t & 1) {
      gkk = warp_sum(gkk);
      gkq = warp_sum(gkq);
    }
    if (lane == 0) {
      float b[1];
      load_f32<1>(static_cast<const T*>(a.proj) + static_cast<int64_t>(row0 + t) * a.ld + a.b_off + h, b);
      *reinterpret_cast<float4*>(out.sc_row(h, row0 + t)) = make_float4(sigmoid_f32(b[0]), qk * rq * rk, gkk, gkq);
    }
  }
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
    if (c >= e) continue;
    float v[TT][VEC];
    conv_rows<T, VEC, TAPS, TT>(src, cr, row0, n, 2 * ck + h * e + c, true, v);
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      if (t >= n) break;
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[t][i] = silu_f32(v[t][i]);
      store_f32<VEC>(out.v_row(h, c / kCols, row0 + t) + c % kCols, v[t]);
    }
  }
}

template <typename T, int VEC, int NJ, int TAPS, int TT>
int launch_prep(const B2DeltaArgs& a, const B2SeqRows& s, bool one_row_each, Status* status, cudaStream_t stream) {
  const int tiles = one_row_each ? s.seqs : (s.rows + TT - 1) / TT + s.seqs;      // every sequence may end in a partial tile
  launch_pdl(delta_prep_kernel<T, VEC, NJ, TAPS, TT>, dim3(tiles, (a.heads + 3) / 4), dim3(128), 0, stream, a, s, prepared_of(a, s.rows), status);
  return last_launch_rc();
}

template <typename T>
int dispatch_prep(const B2DeltaArgs& a, const B2SeqRows& s, bool one_row_each, Status* status, cudaStream_t stream) {
  const int m = a.dim > a.vdim ? a.dim : a.vdim;
  if (a.taps == 4 && a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ld % 4 == 0 && a.ld_dg % 4 == 0) {
    if (m <= 128)
      return one_row_each ? launch_prep<T, 4, 1, 4, 1>(a, s, true, status, stream) : launch_prep<T, 4, 1, 4, 4>(a, s, false, status, stream);
    return launch_prep<T, 4, 2, 4, 2>(a, s, one_row_each, status, stream);
  }
  return launch_prep<T, 1, 8, 0, 2>(a, s, one_row_each, status, stream);
}

// ------------------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------------------
// Thread (rg, cg): columns [cg * VEC, + VEC), key rows rg + i * n_rg. RPT > 0: they stay in registers between the two uses;
// RPT == 0 (states too large, or vdim no multiple of 4): they are read twice.
template <typename T, int VEC, int RPT, int THREADS>
__global__ void __launch_bounds__(THREADS, RPT == 16 ? 3 : 1) delta_decode_kernel(const B2DeltaArgs a, const B2SeqRows sq, const Prepared in, int n_cg, int n_rg,
                                                               Status* status) {
  ptx::grid_dep_sync();
  __shared__ __align__(16) float qkg[3 * kMaxDim];
  __shared__ __align__(16) float red_k[THREADS * VEC], red_q[THREADS * VEC];
  __shared__ float scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int d = a.dim, e = a.vdim;
  const int row = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (row < 0 || row >= sq.rows || !cr.load(sq, seq, row, sq.banks, status)) return;      // uniform per CTA
  if (!B2_ASSERT(status, cr.end == row + 1, kSiteKvIndex, row, cr.end)) return;
  const int cg = tid % n_cg, rg = tid / n_cg;
  const bool active = rg < n_rg;
  float* S = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e + cg * VEC;
  constexpr bool kHeld = RPT > 0;
  float st[kHeld ? RPT : 1][VEC];
  const auto fetch = [&](int r, float (&x)[VEC]) {
#pragma unroll
    for (int v = 0; v < VEC; ++v) x[v] = 0.0f;
    if (active && r < d && cr.rd >= 0) load_f32<VEC>(S + static_cast<int64_t>(r) * e, x);
  };
  const int passes = kHeld ? RPT : (d + n_rg - 1) / n_rg;
  if constexpr (kHeld) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) fetch(rg + i * n_rg, st[i]);
  }
  const float* src = in.qkg_row(h, row);
  for (int i = tid * 4; i < 3 * in.kd; i += THREADS * 4) *reinterpret_cast<float4*>(qkg + i) = *reinterpret_cast<const float4*>(src + i);
  const float4 sc = *reinterpret_cast<const float4*>(in.sc_row(h, row));      // beta, k . q
  float v_in[VEC];
#pragma unroll
  for (int v = 0; v < VEC; ++v) v_in[v] = 0.0f;
  if (active) load_f32<VEC>(in.v_row(h, cg * VEC / kCols, row) + cg * VEC % kCols, v_in);
  __syncthreads();
  const float *q_sm = qkg, *k_sm = qkg + in.kd, *g_sm = qkg + 2 * in.kd;
  if (active) {
    float ks[VEC], qs[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) ks[v] = qs[v] = 0.0f;
#pragma unroll
    for (int i = 0; i < passes; ++i) {
      const int r = rg + i * n_rg;
      if (r < d) {
        const float g = g_sm[r], kr = k_sm[r], qr = q_sm[r];
        float (&x)[VEC] = st[kHeld ? i : 0];
        if constexpr (!kHeld) fetch(r, x);
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          x[v] *= g;
          ks[v] = fmaf(x[v], kr, ks[v]);
          qs[v] = fmaf(x[v], qr, qs[v]);
        }
      }
    }
    store_f32<VEC>(red_k + rg * e + cg * VEC, ks);
    store_f32<VEC>(red_q + rg * e + cg * VEC, qs);
  }
  __syncthreads();
  // every thread sums its own columns, so the write needs no second barrier
  float u[VEC], o[VEC];
#pragma unroll
  for (int v = 0; v < VEC; ++v) u[v] = o[v] = 0.0f;
  if (active) {
    for (int i = 0; i < n_rg; ++i) {
      float x[VEC];
      load_f32<VEC>(red_k + i * e + cg * VEC, x);
#pragma unroll
      for (int v = 0; v < VEC; ++v) u[v] += x[v];
    }
#pragma unroll
    for (int v = 0; v < VEC; ++v) u[v] = sc.x * (v_in[v] - u[v]);
#pragma unroll
    for (int i = 0; i < passes; ++i) {
      const int r = rg + i * n_rg;
      if (r < d) {
        const float kr = k_sm[r];
        float (&x)[VEC] = st[kHeld ? i : 0];
        if constexpr (!kHeld) {
          fetch(r, x);
#pragma unroll
          for (int v = 0; v < VEC; ++v) x[v] *= g_sm[r];
        }
#pragma unroll
        for (int v = 0; v < VEC; ++v) x[v] = fmaf(kr, u[v], x[v]);
        store_f32<VEC>(S + static_cast<int64_t>(r) * e, x);
      }
    }
  }
  float ss = 0.0f;
  if (rg == 0) {
    for (int i = 0; i < n_rg; ++i) {
      float x[VEC];
      load_f32<VEC>(red_q + i * e + cg * VEC, x);
#pragma unroll
      for (int v = 0; v < VEC; ++v) o[v] += x[v];
    }
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
      o[v] = fmaf(u[v], sc.y, o[v]);
      ss = fmaf(o[v], o[v], ss);
    }
  }
  ss = block_sum(ss, scratch);
  if (rg == 0) {
    const float r_o = 1.0f / sqrtf(ss / static_cast<float>(e) + a.eps);
    float z[VEC], w[VEC];
    load_f32<VEC>(static_cast<const T*>(a.dg) + static_cast<int64_t>(row) * a.ld_dg + a.heads * d + h * e + cg * VEC, z);
    load_f32<VEC>(a.norm_w + cg * VEC, w);
#pragma unroll
    for (int v = 0; v < VEC; ++v) o[v] = o[v] * r_o * w[v] * sigmoid_f32(z[v]);
    store_f32<VEC>(static_cast<T*>(a.out) + static_cast<int64_t>(row) * a.ld_out + static_cast<int64_t>(h) * e + cg * VEC, o);
  }
}

template <typename T, int VEC, int RPT>
int launch_decode(const B2DeltaArgs& a, const B2SeqRows& s, int n, int n_cg, int n_rg, Status* status, cudaStream_t stream) {
  constexpr int kThreads = 256;
  launch_pdl(delta_decode_kernel<T, VEC, RPT, kThreads>, dim3(a.heads, n), dim3(kThreads), 0, stream, a, s, prepared_of(a, s.rows), n_cg, n_rg, status);
  return last_launch_rc();
}

template <typename T>
int dispatch_decode(const B2DeltaArgs& a, const B2SeqRows& s, int n, Status* status, cudaStream_t stream) {
  const bool v4 = a.vdim % 4 == 0 && a.ld_dg % 4 == 0 && a.ld_out % 4 == 0 && (a.heads * a.dim) % 4 == 0;
  const int n_cg = v4 ? a.vdim / 4 : a.vdim;
  int n_rg = 256 / n_cg;
  if (n_rg > a.dim) n_rg = a.dim;
  if (!v4) return launch_decode<T, 1, 0>(a, s, n, n_cg, n_rg, status, stream);
  const int rpt = (a.dim + n_rg - 1) / n_rg;
  if (rpt <= 2) return launch_decode<T, 4, 2>(a, s, n, n_cg, n_rg, status, stream);
  if (rpt <= 4) return launch_decode<T, 4, 4>(a, s, n, n_cg, n_rg, status, stream);
  if (rpt <= 8) return launch_decode<T, 4, 8>(a, s, n, n_cg, n_rg, status, stream);
  if (rpt <= 16) return launch_decode<T, 4, 16>(a, s, n, n_cg, n_rg, status, stream);
  if (rpt <= 32) return launch_decode<T, 4, 32>(a, s, n, n_cg, n_rg, status, stream);
  return launch_decode<T, 4, 0>(a, s, n, n_cg, n_rg, status, stream);
}

// ------------------------------------------------------------------------------------------------------------
// scan
// ------------------------------------------------------------------------------------------------------------
// Packed pairs of f32 (two key rows): one instruction per two multiply-adds.
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ float half_sum(uint64_t v) {
  const float2 f = unpack2(v);
  return f.x + f.y;
}

// P pairs of key rows per lane (kd = 32 P). One shared-memory stage: qkg [16][3][kd], v [16][32], sc [16][4].
template <int P>
struct ScanLayout {
  static constexpr int kD = 32 * P;
  static constexpr int kQkg = kTile * 3 * kD, kV = kTile * kCols, kSc = kTile * 4;
  static constexpr int kStage = kQkg + kV + kSc;                 // floats
  static constexpr int kNeutral = 3 * kD + kCols + 4;            // one row that changes nothing, behind the stages
  static constexpr int kBytes = (kStages * kStage + kNeutral) * 4 + kStages * 8;
};

// The pairs of key rows of lane group rg: pair p of P covers rows pair_row(p), pair_row(p) + 1.
template <int P>
__device__ __forceinline__ int pair_row(int p, int rg) {
  if constexpr (P == 1) return 2 * rg;
  else return (p >> 1) * 64 + rg * 4 + (p & 1) * 2;
}
template <int P>
__device__ __forceinline__ void load_pairs(const float* x, int rg, uint64_t (&v)[P]) {
  if constexpr (P == 1) {
    v[0] = *reinterpret_cast<const uint64_t*>(x + 2 * rg);
  } else {
#pragma unroll
    for (int i = 0; i < P / 2; ++i) {
      const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(x + i * 64 + rg * 4);
      v[2 * i] = t.x;
      v[2 * i + 1] = t.y;
    }
  }
}

// Lane (rg = lane & 15, half = lane >> 4) of warp w: value columns col0 + (2 w + half) * 4 + 0..3, P pairs of key rows.
template <int P>
__global__ void __launch_bounds__(128) delta_scan_kernel(const B2DeltaArgs a, const B2SeqRows sq, const Prepared in, int first, Status* status) {
  ptx::grid_dep_sync();
  using L = ScanLayout<P>;
  extern __shared__ __align__(128) float scan_sm[];
  const int seq = first + blockIdx.z, h = blockIdx.y, blk = blockIdx.x, col0 = blk * kCols;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int begin = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (sq.seq_rows[2 * seq + 1] <= begin || !cr.load(sq, seq, begin, sq.banks, status)) return;      // uniform per CTA
  const int d = a.dim, e = a.vdim, n = cr.end - cr.begin;
  const int n_tiles = (n + kTile - 1) / kTile;
  float* neutral = scan_sm + kStages * L::kStage;
  const uint32_t bars = ptx::smem_u32(neutral + L::kNeutral);
  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) ptx::mbar_init(bars + 8 * s, 1);
    ptx::fence_mbar_init();
  }
  for (int i = threadIdx.x; i < L::kNeutral; i += 128) neutral[i] = i >= 2 * L::kD && i < 3 * L::kD ? 1.0f : 0.0f;
  __syncthreads();
  const auto issue = [&](int i) {      // thread 0: start the copies of tile i
    const int rows = min(kTile, n - i * kTile), row = begin + i * kTile;
    float* st = scan_sm + (i % kStages) * L::kStage;
    const uint32_t bar = bars + 8 * (i % kStages);
    ptx::mbar_arrive_expect_tx(bar, static_cast<uint32_t>(rows * (3 * L::kD + kCols + 4) * 4));
    ptx::bulk_load(ptx::smem_u32(st), in.qkg_row(h, row), rows * 3 * L::kD * 4, bar);
    ptx::bulk_load(ptx::smem_u32(st + L::kQkg), in.v_row(h, blk, row), rows * kCols * 4, bar);
    ptx::bulk_load(ptx::smem_u32(st + L::kQkg + L::kV), in.sc_row(h, row), rows * 16, bar);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < kStages - 1 && i < n_tiles; ++i) issue(i);

  const int rg = lane & 15, c4 = (2 * warp + (lane >> 4)) * 4, base_lane = lane & 16;
  const bool b3 = lane & 8, b2_ = lane & 4, b1 = lane & 2, b0 = lane & 1;
  const int my_col = lane & 3;      // after the reduction a lane holds one sum: kind (S^T k, S^T q) = bit 3, row = bit 2, column = bits 1, 0
  float* state = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e + col0 + c4;
  uint64_t S[P][4];
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int key = pair_row<P>(p, rg);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      float lo = 0.0f, hi = 0.0f;
      if (cr.rd >= 0 && col0 + c4 + c < e) {
        if (key < d) lo = state[static_cast<int64_t>(key) * e + c];
        if (key + 1 < d) hi = state[static_cast<int64_t>(key + 1) * e + c];
      }
      S[p][c] = pack2(lo, hi);
    }
  }
  const int64_t o_ld = static_cast<int64_t>(a.heads) * e;
  float* o_dst = a.o_raw + static_cast<int64_t>(begin + (b2_ ? 1 : 0)) * o_ld + static_cast<int64_t>(h) * e + col0 + c4 + my_col;
  const bool writes = b3 && col0 + c4 + my_col < e;
  bool failed = false;
  for (int i = 0; i < n_tiles; ++i) {
    // the stage of tile i - 1 was released by the barrier at the end of that tile
    if (threadIdx.x == 0 && i + kStages - 1 < n_tiles) issue(i + kStages - 1);
    if (!ptx::mbar_wait(bars + 8 * (i % kStages), (i / kStages) & 1)) {
      status_record(status, kTimeout, kSiteAttn, seq, i);
      failed = true;
    }
    const float* st = scan_sm + (i % kStages) * L::kStage;
    const int rows = min(kTile, n - i * kTile);
#pragma unroll 1
    for (int t = 0; t < rows; t += 2) {
      const bool two = t + 1 < rows;
      const float* t1 = st + t * 3 * L::kD;
      const float* t2 = two ? t1 + 3 * L::kD : neutral;
      const float* v1 = st + L::kQkg + t * kCols + c4;
      const float* v2 = two ? v1 + kCols : neutral + 3 * L::kD;
      const float4 sc1 = *reinterpret_cast<const float4*>(st + L::kQkg + L::kV + t * 4);
      const float4 sc2 = *reinterpret_cast<const float4*>(two ? st + L::kQkg + L::kV + t * 4 + 4 : neutral + 3 * L::kD + kCols);
      uint64_t q1[P], k1[P], g1[P], q2[P], k2[P], g2[P];
      load_pairs<P>(t1, rg, q1);
      load_pairs<P>(t1 + L::kD, rg, k1);
      load_pairs<P>(t1 + 2 * L::kD, rg, g1);
      load_pairs<P>(t2, rg, q2);
      load_pairs<P>(t2 + L::kD, rg, k2);
      load_pairs<P>(t2 + 2 * L::kD, rg, g2);
      uint64_t acc[4][4];      // [S1 k1, S1 q1 | S2 k2, S2 q2] per column, even and odd rows apart
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[j][c] = 0;
#pragma unroll
      for (int p = 0; p < P; ++p) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          S[p][c] = mul2(S[p][c], g1[p]);
          acc[0][c] = fma2(S[p][c], k1[p], acc[0][c]);
          acc[1][c] = fma2(S[p][c], q1[p], acc[1][c]);
          S[p][c] = mul2(S[p][c], g2[p]);
          acc[2][c] = fma2(S[p][c], k2[p], acc[2][c]);
          acc[3][c] = fma2(S[p][c], q2[p], acc[3][c]);
        }
        k1[p] = mul2(k1[p], g2[p]);      // the first row's write, decayed by the second row
      }
      // sum over the 16 lane groups, halving the values per lane: kind, row, then two bits of the column
      float x8[8], x4[4], x2[2], x;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const float sk1 = half_sum(acc[0][c]), sq1 = half_sum(acc[1][c]), sk2 = half_sum(acc[2][c]), sq2 = half_sum(acc[3][c]);
        x8[c] = (b3 ? sq1 : sk1) + __shfl_xor_sync(0xffffffffu, b3 ? sk1 : sq1, 8);
        x8[4 + c] = (b3 ? sq2 : sk2) + __shfl_xor_sync(0xffffffffu, b3 ? sk2 : sq2, 8);
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) x4[c] = (b2_ ? x8[4 + c] : x8[c]) + __shfl_xor_sync(0xffffffffu, b2_ ? x8[c] : x8[4 + c], 4);
#pragma unroll
      for (int c = 0; c < 2; ++c) x2[c] = (b1 ? x4[2 + c] : x4[c]) + __shfl_xor_sync(0xffffffffu, b1 ? x4[c] : x4[2 + c], 2);
      x = (b0 ? x2[1] : x2[0]) + __shfl_xor_sync(0xffffffffu, b0 ? x2[0] : x2[1], 1);
      const float u1_own = sc1.x * (v1[my_col] - x);                                              // right where bits 3, 2 are clear
      const float u1s = __shfl_sync(0xffffffffu, u1_own, base_lane + my_col);                     // row 1's u of this lane's column
      const float u2_own = sc2.x * (v2[my_col] - fmaf(u1s, sc2.z, x));                            // right where bit 3 is clear, bit 2 set
      float u1[4], u2[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        u1[c] = __shfl_sync(0xffffffffu, u1_own, base_lane + c);
        u2[c] = __shfl_sync(0xffffffffu, u2_own, base_lane + 4 + c);
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const uint64_t w1 = pack2(u1[c], u1[c]), w2 = pack2(u2[c], u2[c]);
#pragma unroll
        for (int p = 0; p < P; ++p) S[p][c] = fma2(k2[p], w2, fma2(k1[p], w1, S[p][c]));
      }
      const float u2s = b1 ? (b0 ? u2[3] : u2[2]) : (b0 ? u2[1] : u2[0]);
      const float o = b2_ ? fmaf(u2s, sc2.y, fmaf(u1s, sc2.w, x)) : fmaf(u1s, sc1.y, x);
      if (writes && (two || !b2_)) o_dst[static_cast<int64_t>(i * kTile + t) * o_ld] = o;
    }
    if (__syncthreads_or(failed)) break;      // also releases the stage
  }
  if (failed) {
    // let copies in flight land before the CTA's shared memory is released
    for (int s = 0; s < kStages; ++s) ptx::mbar_wait(bars + 8 * s, 0, 20000000ull) || ptx::mbar_wait(bars + 8 * s, 1, 20000000ull);
    return;
  }
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int key = pair_row<P>(p, rg);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      if (col0 + c4 + c >= e) continue;
      const float2 f = unpack2(S[p][c]);
      if (key < d) state[static_cast<int64_t>(key) * e + c] = f.x;
      if (key + 1 < d) state[static_cast<int64_t>(key + 1) * e + c] = f.y;
    }
  }
}

// out = rms_norm(o) * w * sigmoid(gate) for the rows of sequences >= first: one warp per (row, head).
template <typename T, int VEC, int NJ>
__global__ void __launch_bounds__(256) delta_out_kernel(const B2DeltaArgs a, const B2SeqRows sq, int first) {
  ptx::grid_dep_sync();
  const int64_t idx = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, e = a.vdim;
  const int row = static_cast<int>(idx / a.heads), h = static_cast<int>(idx % a.heads);
  if (row >= sq.rows || sq.row_seq[row] < first) return;
  const float* o = a.o_raw + (static_cast<int64_t>(row) * a.heads + h) * e;
  const T* gate = static_cast<const T*>(a.dg) + static_cast<int64_t>(row) * a.ld_dg + a.heads * a.dim + h * e;
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(row) * a.ld_out + static_cast<int64_t>(h) * e;
  float v[NJ][VEC], ss = 0.0f;
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[j][i] = 0.0f;
    if (c < e) load_f32<VEC>(o + c, v[j]);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[j][i], v[j][i], ss);
  }
  ss = warp_sum(ss);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(e) + a.eps);
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
    if (c >= e) continue;
    float z[VEC], w[VEC];
    load_f32<VEC>(gate + c, z);
    load_f32<VEC>(a.norm_w + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[j][i] = v[j][i] * r * w[i] * sigmoid_f32(z[i]);
    store_f32<VEC>(out + c, v[j]);
  }
}

template <int P>
int launch_scan(const B2DeltaArgs& a, const B2SeqRows& s, int first, int n, Status* status, cudaStream_t stream) {
  using L = ScanLayout<P>;
  static DeviceOnce attr_once;
  if (const int rc = attr_once.max_smem(delta_scan_kernel<P>, L::kBytes)) return rc;
  launch_pdl(delta_scan_kernel<P>, dim3((a.vdim + kCols - 1) / kCols, a.heads, n), dim3(128), L::kBytes, stream, a, s, prepared_of(a, s.rows), first, status);
  return last_launch_rc();
}

int dispatch_scan(const B2DeltaArgs& a, const B2SeqRows& s, int first, int n, Status* status, cudaStream_t stream) {
  switch (padded_dim(a.dim)) {
    case 32: return launch_scan<1>(a, s, first, n, status, stream);
    case 64: return launch_scan<2>(a, s, first, n, status, stream);
    case 128: return launch_scan<4>(a, s, first, n, status, stream);
    default: return launch_scan<8>(a, s, first, n, status, stream);
  }
}

template <typename T>
int run_delta(const B2DeltaArgs& a, const B2SeqRows& s, int n_decode, int first, int n_prefill, Status* status, cudaStream_t stream) {
  if (const int rc = dispatch_prep<T>(a, s, n_prefill == 0, status, stream)) return rc;
  if (n_decode > 0)
    if (const int rc = dispatch_decode<T>(a, s, n_decode, status, stream)) return rc;
  if (n_prefill == 0) return 0;
  if (const int rc = dispatch_scan(a, s, first, n_prefill, status, stream)) return rc;
  const dim3 grid(static_cast<unsigned>((static_cast<int64_t>(s.rows) * a.heads + 7) / 8));
  const bool v4 = a.vdim % 4 == 0 && a.ld_dg % 4 == 0 && a.ld_out % 4 == 0 && (a.heads * a.dim) % 4 == 0;
  if (v4 && a.vdim <= 128) launch_pdl(delta_out_kernel<T, 4, 1>, grid, dim3(256), 0, stream, a, s, first);
  else if (v4) launch_pdl(delta_out_kernel<T, 4, 2>, grid, dim3(256), 0, stream, a, s, first);
  else launch_pdl(delta_out_kernel<T, 1, 8>, grid, dim3(256), 0, stream, a, s, first);
  return last_launch_rc();
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int64_t b2_delta_scratch_floats(int heads, int dim, int vdim, int rows) { return scratch_floats(heads, dim, vdim, rows); }

extern "C" int b2_delta_rule(const B2DeltaArgs* a, const B2SeqRows* s, int n_decode, int first, int n_prefill, int f32, Status* status,
                             cudaStream_t stream) {
  if (s->rows <= 0 || n_decode + n_prefill <= 0) return 0;
  if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads != 0 || a->heads > 65535 || a->dim <= 0 || a->dim > kMaxDim || a->vdim <= 0 ||
      a->vdim > kMaxDim || a->taps < 1 || (a->taps > 1 && a->conv_state == nullptr) || a->state == nullptr || a->out == nullptr ||
      a->scratch == nullptr || a->ld_out < static_cast<int64_t>(a->heads) * a->vdim || n_decode < 0 || n_prefill < 0 || first < n_decode ||
      first + n_prefill > s->seqs || n_decode > 65535 || n_prefill > 65535 || (n_prefill > 0 && a->o_raw == nullptr))
    return -kBadArgument;
  return f32 ? run_delta<float>(*a, *s, n_decode, first, n_prefill, status, stream)
             : run_delta<__nv_bfloat16>(*a, *s, n_decode, first, n_prefill, status, stream);
}
