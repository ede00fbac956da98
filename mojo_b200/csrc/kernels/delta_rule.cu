// Gated delta rule with one decay per key channel. State S [dim, vdim] per head, all of it in f32:
//   S <- g * S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q
// Both kernels read S^T k and S^T q off the decayed state together and add the new write's share u (k . q) to the output,
// so a token costs one pass over S and one reduction. The projections come in raw: short convolution, silu, unit norms,
// decays and step sizes are computed where they are used.
//   decode: one row per sequence. CTA = (head, sequence); S streams through registers once; output norm and gate fused.
//   scan:   any number of rows. CTA = (32 value columns, head, sequence); four warps keep their part of S in registers and
//           walk over the rows, four other warps prepare the next rows' q, k, g, v in shared memory meanwhile.
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

__device__ __forceinline__ float silu_f32(float x) { return x / (1.0f + expf(-x)); }

// ------------------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------------------
// Thread (rg, cg): columns [cg * VEC, + VEC), rows rg + i * RG. THREADS / (vdim / VEC) row groups.
template <typename T, int VEC, int RPT, int THREADS>
__global__ void __launch_bounds__(THREADS) delta_decode_kernel(const B2DeltaArgs a, const B2SeqRows sq, int n_cg, int n_rg, Status* status) {
  ptx::grid_dep_sync();
  __shared__ float q_sm[kMaxDim], k_sm[kMaxDim], g_sm[kMaxDim], v_sm[kMaxDim], u_sm[kMaxDim];
  __shared__ float red_k[THREADS * VEC], red_q[THREADS * VEC];
  __shared__ float norms[3];           // |q|^2, |k|^2, q . k of the raw vectors
  __shared__ float scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int d = a.dim, e = a.vdim;
  const int row = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (row < 0 || row >= sq.rows || !cr.load(sq, seq, row, sq.banks, status)) return;      // uniform per CTA
  if (!B2_ASSERT(status, cr.end == row + 1, kSiteKvIndex, row, cr.end)) return;
  const int per = a.heads / a.kv_heads, kh = h / per;
  const int cg = tid % n_cg, rg = tid / n_cg;
  const bool active = rg < n_rg;
  float* S = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e;

  // the state is on its way while the small vectors are prepared
  float st[RPT][VEC];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = rg + i * n_rg;
#pragma unroll
    for (int v = 0; v < VEC; ++v) st[i][v] = 0.0f;
    if (active && r < d && cr.rd >= 0) load_f32<VEC>(S + static_cast<int64_t>(r) * e + cg * VEC, st[i]);
  }
  const int ck = a.kv_heads * d;         // channels: q | k | v
  const int channels = 2 * ck + a.heads * e;
  const ConvSource<T> src{static_cast<const T*>(a.proj), a.ld, a.conv_w, static_cast<T*>(a.conv_state), a.taps, channels, sq.banks};
  const T* dg = static_cast<const T*>(a.dg) + static_cast<int64_t>(row) * a.ld_dg;
  for (int i = tid; i < 2 * d + e; i += THREADS) {
    const bool is_v = i >= 2 * d;
    const int chan = is_v ? 2 * ck + h * e + (i - 2 * d) : i < d ? kh * d + i : ck + kh * d + (i - d);
    float y[1];
    src.template apply<1>(cr, row, chan, y);
    if (is_v || h % per == 0) src.template save<1>(cr, row, chan);
    const float s = silu_f32(y[0]);
    if (is_v) v_sm[i - 2 * d] = s;
    else if (i < d) q_sm[i] = s;
    else k_sm[i - d] = s;
  }
  for (int i = tid; i < d; i += THREADS) {
    float z[1];
    load_f32<1>(dg + h * d + i, z);
    g_sm[i] = expf(a.neg_rate[h] * softplus_f32(z[0] + a.dt_bias[h * d + i]));
  }
  __syncthreads();
  if (tid < 96) {                        // three warps, three sums
    const int w = tid >> 5, lane = tid & 31;
    const float* x = w == 1 ? k_sm : q_sm;
    const float* y = w == 0 ? q_sm : k_sm;
    float s = 0.0f;
    for (int i = lane; i < d; i += 32) s = fmaf(x[i], y[i], s);
    s = warp_sum(s);
    if (lane == 0) norms[w] = s;
  }
  __syncthreads();
  const float rq = rsqrtf(static_cast<float>(d)) / sqrtf(norms[0] + kUnitEps), rk = 1.0f / sqrtf(norms[1] + kUnitEps);
  float ks[VEC], qs[VEC];
#pragma unroll
  for (int v = 0; v < VEC; ++v) ks[v] = qs[v] = 0.0f;
  if (active) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = rg + i * n_rg;
      if (r < d) {
        const float g = g_sm[r], kr = k_sm[r], qr = q_sm[r];
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          st[i][v] *= g;
          ks[v] = fmaf(st[i][v], kr, ks[v]);
          qs[v] = fmaf(st[i][v], qr, qs[v]);
        }
      }
    }
    store_f32<VEC>(red_k + rg * e + cg * VEC, ks);
    store_f32<VEC>(red_q + rg * e + cg * VEC, qs);
  }
  __syncthreads();
  float b[1];
  load_f32<1>(static_cast<const T*>(a.proj) + static_cast<int64_t>(row) * a.ld + a.b_off + h, b);
  const float beta = sigmoid_f32(b[0]);
  const float kq = norms[2] * rq * rk;
  float o_sq = 0.0f;
  for (int c = tid; c < e; c += THREADS) {
    float sk = 0.0f, sq2 = 0.0f;
    for (int i = 0; i < n_rg; ++i) {
      sk += red_k[i * e + c];
      sq2 += red_q[i * e + c];
    }
    const float u = beta * (v_sm[c] - sk * rk);
    u_sm[c] = u * rk;                    // S gets k u^T with the unit k: rk goes into u
    const float o = sq2 * rq + u * kq;
    v_sm[c] = o;
    o_sq = fmaf(o, o, o_sq);
  }
  o_sq = block_sum(o_sq, scratch);       // also orders u_sm
  if (active) {
    float u[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) u[v] = u_sm[cg * VEC + v];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = rg + i * n_rg;
      if (r < d) {
#pragma unroll
        for (int v = 0; v < VEC; ++v) st[i][v] = fmaf(k_sm[r], u[v], st[i][v]);
        store_f32<VEC>(S + static_cast<int64_t>(r) * e + cg * VEC, st[i]);
      }
    }
  }
  const float r_o = 1.0f / sqrtf(o_sq / static_cast<float>(e) + a.eps);
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(row) * a.ld_out + static_cast<int64_t>(h) * e;
  for (int c = tid; c < e; c += THREADS) {
    float z[1], y[1];
    load_f32<1>(dg + a.heads * d + h * e + c, z);
    y[0] = v_sm[c] * r_o * a.norm_w[c] * sigmoid_f32(z[0]);
    store_f32<1>(out + c, y);
  }
}

template <typename T, int VEC, int THREADS>
int launch_decode(const B2DeltaArgs& a, const B2SeqRows& s, int n, Status* status, cudaStream_t stream) {
  const int n_cg = a.vdim / VEC;
  if (n_cg > THREADS) return -kBadArgument;
  int n_rg = THREADS / n_cg;
  if (n_rg > a.dim) n_rg = a.dim;
  const int rpt = (a.dim + n_rg - 1) / n_rg;
  const dim3 grid(a.heads, n);
#define B2_DD(R_)                                                                                                             \
  {                                                                                                                           \
    launch_pdl(delta_decode_kernel<T, VEC, R_, THREADS>, grid, dim3(THREADS), 0, stream, a, s, n_cg, n_rg, status);           \
    return last_launch_rc();                                                                                                  \
  }
  if (rpt <= 2) B2_DD(2);
  if (rpt <= 4) B2_DD(4);
  if (rpt <= 8) B2_DD(8);
  if (rpt <= 16) B2_DD(16);
  if constexpr (VEC == 4 && THREADS == 256) {
    if (rpt <= 32) B2_DD(32);
  }
#undef B2_DD
  return -kTooLarge;
}

template <typename T>
int dispatch_decode(const B2DeltaArgs& a, const B2SeqRows& s, int n, Status* status, cudaStream_t stream) {
  // a thread keeps at most 64 (256 threads: 128) state elements
  if (a.vdim % 4 == 0) {
    const int rows256 = (a.dim + 256 / (a.vdim / 4) - 1) / (256 / (a.vdim / 4));
    if (rows256 <= 16 || a.dim * a.vdim <= 32768) return launch_decode<T, 4, 256>(a, s, n, status, stream);
    return launch_decode<T, 4, 1024>(a, s, n, status, stream);
  }
  const int r = launch_decode<T, 1, 256>(a, s, n, status, stream);
  return r == -kTooLarge ? launch_decode<T, 1, 1024>(a, s, n, status, stream) : r;
}

// ------------------------------------------------------------------------------------------------------------
// scan
// ------------------------------------------------------------------------------------------------------------
constexpr int kTile = 16;        // rows prepared at a time
constexpr int kCols = 32;        // value columns per CTA

// Shared-memory row of one token: q [D], k [D], g [D], v [32], beta, k . q (+ padding to a multiple of 4 floats)
template <int R>
struct ScanLayout {
  static constexpr int kD = 16 * R;          // key channels, padded with zero rows
  static constexpr int kTok = 3 * kD + kCols + 4;
  static constexpr int kBytes = 2 * kTile * kTok * 4;
};

template <typename T, int R>
__device__ __forceinline__ void scan_prepare(const B2DeltaArgs& a, const ConvSource<T>& src, const ConvRow& cr, float* tile, int row0, int n_rows,
                                             int h, int col0, bool save_qk, int warp, int lane) {
  using L = ScanLayout<R>;
  constexpr int NJ = (L::kD + 31) / 32;
  const int d = a.dim, e = a.vdim, per = a.heads / a.kv_heads, kh = h / per, ck = a.kv_heads * d;
  const float neg_rate = a.neg_rate[h];
  for (int t = warp; t < n_rows; t += 4) {
    const int row = row0 + t;
    float* dst = tile + t * L::kTok;
    const T* dg = static_cast<const T*>(a.dg) + static_cast<int64_t>(row) * a.ld_dg + h * d;
    float q[NJ], k[NJ], qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int i = lane + 32 * j;
      q[j] = k[j] = 0.0f;
      float g = 1.0f;
      if (i < d) {
        float y[1], z[1];
        src.template apply<1>(cr, row, kh * d + i, y);
        q[j] = silu_f32(y[0]);
        src.template apply<1>(cr, row, ck + kh * d + i, y);
        k[j] = silu_f32(y[0]);
        if (save_qk) {
          src.template save<1>(cr, row, kh * d + i);
          src.template save<1>(cr, row, ck + kh * d + i);
        }
        load_f32<1>(dg + i, z);
        g = expf(neg_rate * softplus_f32(z[0] + a.dt_bias[h * d + i]));
      }
      qq = fmaf(q[j], q[j], qq);
      kk = fmaf(k[j], k[j], kk);
      qk = fmaf(q[j], k[j], qk);
      if (i < L::kD) dst[2 * L::kD + i] = g;
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    qk = warp_sum(qk);
    const float rq = rsqrtf(static_cast<float>(d)) / sqrtf(qq + kUnitEps), rk = 1.0f / sqrtf(kk + kUnitEps);
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int i = lane + 32 * j;
      if (i < L::kD) {
        dst[i] = q[j] * rq;
        dst[L::kD + i] = k[j] * rk;
      }
    }
    float v = 0.0f;
    if (col0 + lane < e) {
      float y[1];
      const int chan = 2 * ck + h * e + col0 + lane;
      src.template apply<1>(cr, row, chan, y);
      src.template save<1>(cr, row, chan);
      v = silu_f32(y[0]);
    }
    dst[3 * L::kD + lane] = v;
    if (lane == 0) {
      float b[1];
      load_f32<1>(static_cast<const T*>(a.proj) + row * a.ld + a.b_off + h, b);
      dst[3 * L::kD + kCols] = sigmoid_f32(b[0]);
      dst[3 * L::kD + kCols + 1] = qk * rq * rk;
    }
  }
}

// Lane (rg = lane & 15, ch = lane >> 4) of consumer warp w: value columns col0 + (2 w + ch) * 4 + 0..3, key rows
// 64 c + 4 rg + 0..3 for c < R / 4.
template <typename T, int R>
__global__ void __launch_bounds__(256) delta_scan_kernel(const B2DeltaArgs a, const B2SeqRows sq, int first, Status* status) {
  ptx::grid_dep_sync();
  using L = ScanLayout<R>;
  extern __shared__ __align__(16) float scan_sm[];
  const int seq = first + blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kCols;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int begin = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (sq.seq_rows[2 * seq + 1] <= begin || !cr.load(sq, seq, begin, sq.banks, status)) return;      // uniform per CTA
  const int d = a.dim, e = a.vdim, n = cr.end - cr.begin;
  const int n_tiles = (n + kTile - 1) / kTile;
  float* tiles[2] = {scan_sm, scan_sm + kTile * L::kTok};
  float* state = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e;

  if (warp >= 4) {
    const int channels = 2 * a.kv_heads * d + a.heads * e;
    const ConvSource<T> src{static_cast<const T*>(a.proj), a.ld, a.conv_w, static_cast<T*>(a.conv_state), a.taps, channels, sq.banks};
    const bool save_qk = blockIdx.x == 0 && h % (a.heads / a.kv_heads) == 0;
    for (int i = 0; i <= n_tiles; ++i) {
      if (i < n_tiles)
        scan_prepare<T, R>(a, src, cr, tiles[i & 1], begin + i * kTile, min(kTile, n - i * kTile), h, col0, save_qk, warp - 4, lane);
      __syncthreads();
    }
    return;
  }

  const int rg = lane & 15, c4 = (2 * warp + (lane >> 4)) * 4;
  const bool b3 = lane & 8, b2_ = lane & 4, b1 = lane & 2;
  const int my_col = (b2_ ? 2 : 0) + (b1 ? 1 : 0);      // the column (of this lane's four) whose sum ends up here
  const int base_lane = lane & 16;
  float S[R][4];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int key = (r >> 2) * 64 + rg * 4 + (r & 3);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      S[r][c] = 0.0f;
      if (cr.rd >= 0 && key < d && col0 + c4 + c < e) S[r][c] = state[static_cast<int64_t>(key) * e + col0 + c4 + c];
    }
  }
  float* o_dst = a.o_raw + static_cast<int64_t>(begin) * a.heads * e + static_cast<int64_t>(h) * e + col0 + c4 + my_col;
  const bool writes = b3 && !(lane & 1) && col0 + c4 + my_col < e;
  __syncthreads();
  for (int i = 0; i < n_tiles; ++i) {
    const float* tile = tiles[i & 1];
    const int rows = min(kTile, n - i * kTile);
    for (int t = 0; t < rows; ++t) {
      const float* tok = tile + t * L::kTok;
      float acc[8];
#pragma unroll
      for (int c = 0; c < 8; ++c) acc[c] = 0.0f;
      float kr[R];
#pragma unroll
      for (int r4 = 0; r4 < R / 4; ++r4) {
        const float4 q4 = *reinterpret_cast<const float4*>(tok + r4 * 64 + rg * 4);
        const float4 k4 = *reinterpret_cast<const float4*>(tok + L::kD + r4 * 64 + rg * 4);
        const float4 g4 = *reinterpret_cast<const float4*>(tok + 2 * L::kD + r4 * 64 + rg * 4);
        const float qv[4] = {q4.x, q4.y, q4.z, q4.w}, gv[4] = {g4.x, g4.y, g4.z, g4.w};
        kr[r4 * 4] = k4.x; kr[r4 * 4 + 1] = k4.y; kr[r4 * 4 + 2] = k4.z; kr[r4 * 4 + 3] = k4.w;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = r4 * 4 + j;
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            S[r][c] *= gv[j];
            acc[c] = fmaf(S[r][c], kr[r], acc[c]);
            acc[4 + c] = fmaf(S[r][c], qv[j], acc[4 + c]);
          }
        }
      }
      // sum over the 16 row groups, halving the values per lane: lanes with bit 3 clear end with the S^T k sums, the
      // others with the S^T q sums; bits 2 and 1 pick the column
      float x4[4], x2[2], x1;
#pragma unroll
      for (int c = 0; c < 4; ++c) x4[c] = (b3 ? acc[4 + c] : acc[c]) + __shfl_xor_sync(0xffffffffu, b3 ? acc[c] : acc[4 + c], 8);
#pragma unroll
      for (int c = 0; c < 2; ++c) x2[c] = (b2_ ? x4[2 + c] : x4[c]) + __shfl_xor_sync(0xffffffffu, b2_ ? x4[c] : x4[2 + c], 4);
      x1 = (b1 ? x2[1] : x2[0]) + __shfl_xor_sync(0xffffffffu, b1 ? x2[0] : x2[1], 2);
      x1 += __shfl_xor_sync(0xffffffffu, x1, 1);
      const float beta = tok[3 * L::kD + kCols];
      const float u_own = beta * (tok[3 * L::kD + c4 + my_col] - x1);       // meaningful where bit 3 is clear
      float u[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) u[c] = __shfl_sync(0xffffffffu, u_own, base_lane + 2 * c);
#pragma unroll
      for (int r = 0; r < R; ++r)
#pragma unroll
        for (int c = 0; c < 4; ++c) S[r][c] = fmaf(kr[r], u[c], S[r][c]);
      if (writes) {
        const float um = b2_ ? (b1 ? u[3] : u[2]) : (b1 ? u[1] : u[0]);
        o_dst[static_cast<int64_t>(i * kTile + t) * a.heads * e] = fmaf(um, tok[3 * L::kD + kCols + 1], x1);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int key = (r >> 2) * 64 + rg * 4 + (r & 3);
#pragma unroll
    for (int c = 0; c < 4; ++c)
      if (key < d && col0 + c4 + c < e) state[static_cast<int64_t>(key) * e + col0 + c4 + c] = S[r][c];
  }
}

// out = rms_norm(o) * w * sigmoid(gate) for the rows of sequences >= first: one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) delta_out_kernel(const B2DeltaArgs a, const B2SeqRows sq, int first) {
  ptx::grid_dep_sync();
  const int64_t idx = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, e = a.vdim;
  const int row = static_cast<int>(idx / a.heads), h = static_cast<int>(idx % a.heads);
  if (row >= sq.rows || sq.row_seq[row] < first) return;
  const float* o = a.o_raw + (static_cast<int64_t>(row) * a.heads + h) * e;
  const T* gate = static_cast<const T*>(a.dg) + static_cast<int64_t>(row) * a.ld_dg + a.heads * a.dim + h * e;
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(row) * a.ld_out + static_cast<int64_t>(h) * e;
  float v[kMaxDim / 32], ss = 0.0f;
#pragma unroll
  for (int j = 0; j < kMaxDim / 32; ++j) {
    const int c = lane + 32 * j;
    v[j] = c < e ? o[c] : 0.0f;
    ss = fmaf(v[j], v[j], ss);
  }
  ss = warp_sum(ss);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(e) + a.eps);
#pragma unroll
  for (int j = 0; j < kMaxDim / 32; ++j) {
    const int c = lane + 32 * j;
    if (c < e) {
      float z[1], y[1];
      load_f32<1>(gate + c, z);
      y[0] = v[j] * r * a.norm_w[c] * sigmoid_f32(z[0]);
      store_f32<1>(out + c, y);
    }
  }
}

template <typename T, int R>
int launch_scan(const B2DeltaArgs& a, const B2SeqRows& s, int first, int n, Status* status, cudaStream_t stream) {
  using L = ScanLayout<R>;
  static DeviceOnce attr_once;
  if (const int rc = attr_once.max_smem(delta_scan_kernel<T, R>, L::kBytes)) return rc;
  launch_pdl(delta_scan_kernel<T, R>, dim3((a.vdim + kCols - 1) / kCols, a.heads, n), dim3(256), L::kBytes, stream, a, s, first, status);
  if (const int rc = last_launch_rc()) return rc;
  const int64_t warps = static_cast<int64_t>(s.rows) * a.heads;
  launch_pdl(delta_out_kernel<T>, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, stream, a, s, first);
  return last_launch_rc();
}

template <typename T>
int dispatch_scan(const B2DeltaArgs& a, const B2SeqRows& s, int first, int n, Status* status, cudaStream_t stream) {
  if (a.dim <= 64) return launch_scan<T, 4>(a, s, first, n, status, stream);
  if (a.dim <= 128) return launch_scan<T, 8>(a, s, first, n, status, stream);
  return launch_scan<T, 16>(a, s, first, n, status, stream);
}

bool delta_args_ok(const B2DeltaArgs& a, const B2SeqRows& s, int first, int n) {
  return a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.dim <= kMaxDim && a.vdim > 0 && a.vdim <= kMaxDim &&
         a.taps >= 1 && (a.taps == 1 || a.conv_state != nullptr) && a.state != nullptr && a.out != nullptr && a.ld_out >= static_cast<int64_t>(a.heads) * a.vdim && first >= 0 && first + n <= s.seqs;
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_delta_decode(const B2DeltaArgs* a, const B2SeqRows* s, int n, int f32, Status* status, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (!delta_args_ok(*a, *s, 0, n) || n > 65535) return -kBadArgument;
  return f32 ? dispatch_decode<float>(*a, *s, n, status, stream) : dispatch_decode<__nv_bfloat16>(*a, *s, n, status, stream);
}

extern "C" int b2_delta_scan(const B2DeltaArgs* a, const B2SeqRows* s, int first, int n, int f32, Status* status, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (!delta_args_ok(*a, *s, first, n) || n > 65535 || a->o_raw == nullptr) return -kBadArgument;
  return f32 ? dispatch_scan<float>(*a, *s, first, n, status, stream) : dispatch_scan<__nv_bfloat16>(*a, *s, first, n, status, stream);
}
