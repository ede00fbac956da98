// Gated linear attention with one decay per key channel. State S [dim, vdim] per head, all of it in f32:
//   S <- diag(a) S + k v^T,  o = S^T q
// Unlike the delta rule, nothing read from the state goes back into it, so a row's update does not wait for the reduction of its
// output. Kernels:
//   decode  one row per sequence. CTA = (head, sequence): S streams through registers once; decays, output norm and gate fused
//   prep    rows of prompt chunks: decays and the scaled query, f32, laid out the way the scan reads them
//   scan    CTA = (32 value columns, head, sequence): S stays in the registers of four warps, which walk over the rows four at a
//           time (one reduction over the key rows for all four) while bulk copies bring the next rows into shared memory
//   out     output norm and gate of the scanned rows
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/recurrence.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kMaxDim = 256;
constexpr int kCols = 32;        // value columns of a scan CTA
constexpr int kStages = 3;
constexpr int kThreadsDecode = 256;

// sigmoid(z)^(1 / tau), from the logarithm of the sigmoid
__device__ __forceinline__ float decay_of(float z, float inv_tau) { return expf(-softplus_f32(-z) * inv_tau); }
__device__ __forceinline__ float silu_f32(float z) { return z * sigmoid_f32(z); }

// Prepared rows, f32, head-major so that a run of rows is one contiguous block.
//   vec [heads][rows][3][kd]             a (one past dim), k, q dim^-0.5 (zero past dim)
//   v   [heads][col blocks][rows][32]    zero past vdim
//   o   [rows][heads * vdim]             outputs of the scan
enum RowVec { kA = 0, kK = 1, kQ = 2, kVecs = 3 };
struct Prepared {
  float* vec;
  float* v;
  float* o;
  int kd, blocks, rows;
  __device__ __forceinline__ float* vec_at(int h, int row) const { return vec + (static_cast<int64_t>(h) * rows + row) * kVecs * kd; }
  __device__ __forceinline__ float* v_at(int h, int blk, int row) const { return v + ((static_cast<int64_t>(h) * blocks + blk) * rows + row) * kCols; }
};
int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
int col_blocks(int vdim) { return (vdim + kCols - 1) / kCols; }
Prepared prepared_of(const B2GatedLinearArgs& a, int rows) {
  Prepared p;
  p.kd = padded_dim(a.dim);
  p.blocks = col_blocks(a.vdim);
  p.rows = rows;
  p.vec = a.scratch;
  p.v = p.vec + static_cast<int64_t>(rows) * a.heads * kVecs * p.kd;
  p.o = p.v + static_cast<int64_t>(rows) * a.heads * p.blocks * kCols;
  return p;
}

// One warp per (row, head), for the rows of sequences >= first.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) gated_prep_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, const Prepared out, int first) {
  ptx::grid_dep_sync();
  const int64_t idx = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, row = static_cast<int>(idx / a.heads), h = static_cast<int>(idx % a.heads), d = a.dim, e = a.vdim;
  if (row >= sq.rows || sq.row_seq[row] < first) return;
  const T* src = static_cast<const T*>(a.proj) + row * a.ld;
  const int nk = a.heads * d;
  const float q_scale = 1.0f / sqrtf(static_cast<float>(d));
  float* dst = out.vec_at(h, row);
  for (int c = lane * VEC; c < out.kd; c += 32 * VEC) {
    float q[VEC] = {}, k[VEC] = {}, z[VEC], g[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) g[i] = 1.0f;
    if (c < d) {
      float b[VEC];
      load_f32<VEC>(src + h * d + c, q);
      load_f32<VEC>(src + nk + h * d + c, k);
      load_f32<VEC>(a.z + row * a.ld_z + h * d + c, z);
      load_f32<VEC>(a.decay_bias + h * d + c, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        g[i] = decay_of(z[i] + b[i], a.inv_tau);
        q[i] *= q_scale;
      }
    }
    store_f32<VEC>(dst + kA * out.kd + c, g);
    store_f32<VEC>(dst + kK * out.kd + c, k);
    store_f32<VEC>(dst + kQ * out.kd + c, q);
  }
  for (int c = lane * VEC; c < out.blocks * kCols; c += 32 * VEC) {
    float v[VEC] = {};
    if (c < e) load_f32<VEC>(src + 2 * nk + h * e + c, v);
    store_f32<VEC>(out.v_at(h, c / kCols, row) + c % kCols, v);
  }
}

template <int P>
struct ScanLayout {
  static constexpr int kD = 32 * P;
  static constexpr int kTile = P >= 8 ? 8 : 16;                          // rows of one stage
  static constexpr int kVec = kVecs * kD;
  static constexpr int kOffV = kTile * kVec;
  static constexpr int kStage = kOffV + kTile * kCols;                   // floats
  static constexpr int kBytes = kStages * kStage * 4 + kStages * 8;
};

// Lane (rg = lane & 15, half = lane >> 4) of warp w: value columns blk * 32 + 8 w + 4 half + 0..3, key rows by pair_row.
template <int P>
__global__ void __launch_bounds__(128) gated_scan_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, const Prepared in, int first, Status* status) {
  ptx::grid_dep_sync();
  using L = ScanLayout<P>;
  extern __shared__ __align__(128) float scan_sm[];
  const int seq = first + blockIdx.z, h = blockIdx.y, blk = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int begin = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (sq.seq_rows[2 * seq + 1] <= begin || !cr.load(sq, seq, begin, sq.banks, status)) return;      // uniform per CTA
  const int d = a.dim, e = a.vdim, n = cr.end - cr.begin, n_tiles = (n + L::kTile - 1) / L::kTile;
  const uint32_t bars = ptx::smem_u32(scan_sm + kStages * L::kStage);
  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) ptx::mbar_init(bars + 8 * s, 1);
    ptx::fence_mbar_init();
  }
  __syncthreads();
  const float *g_vec = in.vec_at(h, begin), *g_v = in.v_at(h, blk, begin);
  const auto issue = [&](int i) {      // thread 0: start the copies of tile i
    const int m = min(L::kTile, n - i * L::kTile);
    const uint32_t st = ptx::smem_u32(scan_sm + (i % kStages) * L::kStage), bar = bars + 8 * (i % kStages);
    ptx::mbar_arrive_expect_tx(bar, static_cast<uint32_t>(m * (L::kVec + kCols) * 4));
    ptx::bulk_load(st, g_vec + static_cast<int64_t>(i) * L::kTile * L::kVec, m * L::kVec * 4, bar);
    ptx::bulk_load(st + L::kOffV * 4, g_v + static_cast<int64_t>(i) * L::kTile * kCols, m * kCols * 4, bar);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < kStages - 1 && i < n_tiles; ++i) issue(i);

  const int rg = lane & 15, c4 = 8 * warp + 4 * (lane >> 4), col = blk * kCols + c4;
  const bool b3 = lane & 8, b2 = lane & 4, b1 = lane & 2, b0 = lane & 1;
  float* state = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e + col;
  uint64_t S[P][4];
  load_state<P>(state, cr.rd < 0, d, e, col, rg, S);
  // after the reduction a lane holds the output of row (lane >> 2) & 3 of the four, column lane & 3
  const int64_t o_ld = static_cast<int64_t>(a.heads) * e;
  const int my_row = (lane >> 2) & 3;
  float* o_dst = in.o + static_cast<int64_t>(begin + my_row) * o_ld + static_cast<int64_t>(h) * e + col + (lane & 3);
  const bool writes = col + (lane & 3) < e;
  bool failed = false;
  for (int i = 0; i < n_tiles; ++i) {
    // the stage of tile i - 1 was released by the barrier at the end of that tile
    if (threadIdx.x == 0 && i + kStages - 1 < n_tiles) issue(i + kStages - 1);
    if (!ptx::mbar_wait(bars + 8 * (i % kStages), (i / kStages) & 1)) {
      status_record(status, kTimeout, kSiteAttn, seq, i);
      failed = true;
    }
    const float* st = scan_sm + (i % kStages) * L::kStage;
    const int m = min(L::kTile, n - i * L::kTile);
#pragma unroll 1
    for (int t0 = 0; t0 < m; t0 += 4) {
      float x[16];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        if (t0 + u < m) {      // uniform
          const float* vec = st + (t0 + u) * L::kVec;
          const float4 v = *reinterpret_cast<const float4*>(st + L::kOffV + (t0 + u) * kCols + c4);
          const uint64_t vv[4] = {pack2(v.x, v.x), pack2(v.y, v.y), pack2(v.z, v.z), pack2(v.w, v.w)};
          uint64_t g[P], k[P], q[P], acc[4];
          load_pairs<P>(vec + kA * L::kD, rg, g);
          load_pairs<P>(vec + kK * L::kD, rg, k);
          load_pairs<P>(vec + kQ * L::kD, rg, q);
#pragma unroll
          for (int p = 0; p < P; ++p)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              S[p][c] = fma2(S[p][c], g[p], mul2(k[p], vv[c]));
              acc[c] = p == 0 ? mul2(S[p][c], q[p]) : fma2(S[p][c], q[p], acc[c]);
            }
#pragma unroll
          for (int c = 0; c < 4; ++c) x[u * 4 + c] = half_sum(acc[c]);
        } else {
#pragma unroll
          for (int c = 0; c < 4; ++c) x[u * 4 + c] = 0.0f;
        }
      }
      float x8[8], x4[4], x2[2];
#pragma unroll
      for (int j = 0; j < 8; ++j) x8[j] = (b3 ? x[8 + j] : x[j]) + __shfl_xor_sync(0xffffffffu, b3 ? x[j] : x[8 + j], 8);
#pragma unroll
      for (int j = 0; j < 4; ++j) x4[j] = (b2 ? x8[4 + j] : x8[j]) + __shfl_xor_sync(0xffffffffu, b2 ? x8[j] : x8[4 + j], 4);
#pragma unroll
      for (int j = 0; j < 2; ++j) x2[j] = (b1 ? x4[2 + j] : x4[j]) + __shfl_xor_sync(0xffffffffu, b1 ? x4[j] : x4[2 + j], 2);
      const float o = (b0 ? x2[1] : x2[0]) + __shfl_xor_sync(0xffffffffu, b0 ? x2[0] : x2[1], 1);
      if (writes && t0 + my_row < m) o_dst[static_cast<int64_t>(i * L::kTile + t0) * o_ld] = o;
    }
    if (__syncthreads_or(failed)) break;      // also releases the stage
  }
  if (failed) {
    // let copies in flight land before the CTA's shared memory is released
    for (int s = 0; s < kStages; ++s) ptx::mbar_wait(bars + 8 * s, 0, 20000000ull) || ptx::mbar_wait(bars + 8 * s, 1, 20000000ull);
    return;
  }
  store_state<P>(state, d, e, col, rg, S);
}

// out = rms_norm(o) * w * silu(gate) * out_scale for the rows of sequences >= first: one warp per (row, head).
template <typename T, int VEC, int NJ>
__global__ void __launch_bounds__(256) gated_out_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, const Prepared in, int first) {
  ptx::grid_dep_sync();
  const int64_t idx = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, e = a.vdim, row = static_cast<int>(idx / a.heads), h = static_cast<int>(idx % a.heads);
  if (row >= sq.rows || sq.row_seq[row] < first) return;
  const float* o = in.o + (static_cast<int64_t>(row) * a.heads + h) * e;
  const T* gate = static_cast<const T*>(a.proj) + row * a.ld + a.heads * (2 * a.dim + e) + h * e;
  T* out = static_cast<T*>(a.out) + row * a.ld_out + static_cast<int64_t>(h) * e;
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
  const float r = a.out_scale / sqrtf(warp_sum(ss) / static_cast<float>(e) + a.eps);
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
    if (c >= e) continue;
    float z[VEC], w[VEC];
    load_f32<VEC>(gate + c, z);
    load_f32<VEC>(a.norm_w + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[j][i] = v[j][i] * r * w[i] * silu_f32(z[i]);
    store_f32<VEC>(out + c, v[j]);
  }
}

// Thread (rg, cg): value columns [cg * VEC, + VEC), key rows rg + i * n_rg, eight of them in flight at a time.
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreadsDecode) gated_decode_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, int n_cg, int n_rg, Status* status) {
  ptx::grid_dep_sync();
  __shared__ __align__(16) float red[kThreadsDecode * VEC];
  __shared__ float vec[kVecs][kMaxDim], scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, d = a.dim, e = a.vdim, nk = a.heads * d;
  ConvRow cr;
  const int row = decode_row(sq, seq, cr, status);
  if (row < 0) return;      // uniform per CTA
  const T* src = static_cast<const T*>(a.proj) + row * a.ld;
  for (int c = threadIdx.x; c < d; c += kThreadsDecode) {
    float q[1], k[1];
    load_f32<1>(src + h * d + c, q);
    load_f32<1>(src + nk + h * d + c, k);
    vec[kA][c] = decay_of(a.z[row * a.ld_z + h * d + c] + a.decay_bias[h * d + c], a.inv_tau);
    vec[kK][c] = k[0];
    vec[kQ][c] = q[0] / sqrtf(static_cast<float>(d));
  }
  const int cg = threadIdx.x % n_cg, rg = threadIdx.x / n_cg;
  const bool active = rg < n_rg, fresh = cr.rd < 0;
  float* S = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e + cg * VEC;
  float v[VEC] = {}, o[VEC] = {};
  if (active) load_f32<VEC>(src + 2 * nk + h * e + cg * VEC, v);
  __syncthreads();
  if (active) {
    for (int r0 = rg; r0 < d; r0 += 8 * n_rg) {
      float x[8][VEC];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = r0 + i * n_rg;
#pragma unroll
        for (int j = 0; j < VEC; ++j) x[i][j] = 0.0f;
        if (r < d && !fresh) load_f32<VEC>(S + static_cast<int64_t>(r) * e, x[i]);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = r0 + i * n_rg;
        if (r >= d) break;
        const float g = vec[kA][r], k = vec[kK][r], q = vec[kQ][r];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          x[i][j] = fmaf(x[i][j], g, k * v[j]);
          o[j] = fmaf(x[i][j], q, o[j]);
        }
        store_f32<VEC>(S + static_cast<int64_t>(r) * e, x[i]);
      }
    }
    store_f32<VEC>(red + rg * e + cg * VEC, o);
  }
  __syncthreads();
  float ss = 0.0f;
  const bool owner = rg == 0;
  if (owner) {
    for (int i = 1; i < n_rg; ++i) {
      float p[VEC];
      load_f32<VEC>(red + i * e + cg * VEC, p);
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] += p[j];
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(o[j], o[j], ss);
  }
  ss = block_sum(ss, scratch);
  if (!owner) return;
  const float r = a.out_scale / sqrtf(ss / static_cast<float>(e) + a.eps);
  float z[VEC], w[VEC];
  load_f32<VEC>(src + 2 * nk + a.heads * e + h * e + cg * VEC, z);
  load_f32<VEC>(a.norm_w + cg * VEC, w);
#pragma unroll
  for (int j = 0; j < VEC; ++j) o[j] = o[j] * r * w[j] * silu_f32(z[j]);
  store_f32<VEC>(static_cast<T*>(a.out) + row * a.ld_out + static_cast<int64_t>(h) * e + cg * VEC, o);
}

template <int P>
int launch_scan(const B2GatedLinearArgs& a, const B2SeqRows& s, int first, int n, Status* status, cudaStream_t stream) {
  using L = ScanLayout<P>;
  static DeviceOnce attr_once;
  if (const int rc = attr_once.max_smem(gated_scan_kernel<P>, L::kBytes)) return rc;
  launch_pdl(gated_scan_kernel<P>, dim3(col_blocks(a.vdim), a.heads, n), dim3(128), L::kBytes, stream, a, s, prepared_of(a, s.rows), first, status);
  return last_launch_rc();
}

template <typename T>
int run_gated(const B2GatedLinearArgs& a, const B2SeqRows& s, int n_decode, int first, int n_prefill, Status* status, cudaStream_t stream) {
  // vector access: every block of a projected row, of the state and of the results begins at a multiple of four elements
  const bool v4 = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ld % 4 == 0 && a.ld_z % 4 == 0 && a.ld_out % 4 == 0 &&
                  ((reinterpret_cast<uintptr_t>(a.proj) | reinterpret_cast<uintptr_t>(a.out)) % (4 * sizeof(T))) == 0 && reinterpret_cast<uintptr_t>(a.z) % 16 == 0;
  if (n_decode > 0) {
    const int n_cg = v4 ? a.vdim / 4 : a.vdim;
    int n_rg = kThreadsDecode / n_cg;
    if (n_rg > a.dim) n_rg = a.dim;
    if (v4) launch_pdl(gated_decode_kernel<T, 4>, dim3(a.heads, n_decode), dim3(kThreadsDecode), 0, stream, a, s, n_cg, n_rg, status);
    else launch_pdl(gated_decode_kernel<T, 1>, dim3(a.heads, n_decode), dim3(kThreadsDecode), 0, stream, a, s, n_cg, n_rg, status);
    if (const int rc = last_launch_rc()) return rc;
  }
  if (n_prefill == 0) return 0;
  const dim3 grid(static_cast<unsigned>((static_cast<int64_t>(s.rows) * a.heads + 7) / 8));
  const Prepared p = prepared_of(a, s.rows);
  if (v4) launch_pdl(gated_prep_kernel<T, 4>, grid, dim3(256), 0, stream, a, s, p, first);
  else launch_pdl(gated_prep_kernel<T, 1>, grid, dim3(256), 0, stream, a, s, p, first);
  if (const int rc = last_launch_rc()) return rc;
  int rc;
  switch (p.kd) {
    case 32: rc = launch_scan<1>(a, s, first, n_prefill, status, stream); break;
    case 64: rc = launch_scan<2>(a, s, first, n_prefill, status, stream); break;
    case 128: rc = launch_scan<4>(a, s, first, n_prefill, status, stream); break;
    default: rc = launch_scan<8>(a, s, first, n_prefill, status, stream);
  }
  if (rc) return rc;
  if (v4 && a.vdim <= 128) launch_pdl(gated_out_kernel<T, 4, 1>, grid, dim3(256), 0, stream, a, s, p, first);
  else if (v4) launch_pdl(gated_out_kernel<T, 4, 2>, grid, dim3(256), 0, stream, a, s, p, first);
  else launch_pdl(gated_out_kernel<T, 1, 8>, grid, dim3(256), 0, stream, a, s, p, first);
  return last_launch_rc();
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int64_t b2_gated_linear_scratch_floats(int heads, int dim, int vdim, int rows) {
  return static_cast<int64_t>(rows) * heads * (kVecs * padded_dim(dim) + col_blocks(vdim) * kCols + vdim);
}

extern "C" int b2_gated_linear(const B2GatedLinearArgs* a, const B2SeqRows* s, int n_decode, int first, int n_prefill, int f32, Status* status,
                               cudaStream_t stream) {
  if (s->rows <= 0 || n_decode + n_prefill <= 0) return 0;
  if (a->heads <= 0 || a->heads > 65535 || a->dim <= 0 || a->dim > kMaxDim || a->vdim <= 0 || a->vdim > kMaxDim || a->state == nullptr || a->out == nullptr ||
      a->ld_out < static_cast<int64_t>(a->heads) * a->vdim || a->ld < 2ll * a->heads * (a->dim + a->vdim) || n_decode < 0 || n_prefill < 0 || first < n_decode ||
      first + n_prefill > s->seqs || n_decode > 65535 || n_prefill > 65535 || (n_prefill > 0 && a->scratch == nullptr))
    return -kBadArgument;
  return f32 ? run_gated<float>(*a, *s, n_decode, first, n_prefill, status, stream)
             : run_gated<__nv_bfloat16>(*a, *s, n_decode, first, n_prefill, status, stream);
}
