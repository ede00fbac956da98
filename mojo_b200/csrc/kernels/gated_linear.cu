// Gated linear attention with one decay per key channel. State S [dim, vdim] per head, all of it in f32:
//   S <- diag(a) S + k v^T,  o = S^T q
// Kernels:
//   decode  one row per sequence. CTA = (head, sequence): S streams through registers once; decays, output norm and gate fused
//   prep    prompt chunks, 16 rows at a time: everything about a block of rows that the state does not enter, see below
//   scan    CTA = (64 value columns, head, sequence): S stays in the registers of four warps, which walk over the blocks while bulk
//           copies bring the next one into shared memory
//   out     the part of a row's output that its own block holds; output norm and gate
// With A_t the product of a block's decays up to row t, R_s the product of those behind row s, and S the state before the block,
//   o_t = S^T (A_t q_t) + sum_{s <= t} P_ts v_s,   P_ts = (q_t . (product of the decays in (s, t]) k_s)
//   S after = diag(A_16) S + sum_s (R_s k_s) v_s^T
// so a block costs two multiply-adds per state element and row instead of three, none of which waits for the row before. All
// products are of factors up to one: nothing is divided by a decay.
// A few long prompts leave most of the machine idle in the scan, which walks over time. Then sequences are cut into segments: a
// first pass finds what every segment adds to the state and how much of the old state it keeps, `carry` combines those into the
// state at every segment's start, and the scan takes all segments at once.
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
constexpr int kBlock = 16;       // rows of a block
constexpr int kCols = 64;        // value columns of a scan CTA
constexpr int kStages = 3;
constexpr int kThreadsDecode = 256;

// sigmoid(z)^(1 / tau), from the logarithm of the sigmoid
__device__ __forceinline__ float decay_of(float z, float inv_tau) { return ptx::ex2(-softplus_fast(-z) * (inv_tau * ptx::kLog2e)); }
__device__ __forceinline__ float silu_f32(float z) { return z * sigmoid_f32(z); }

// Prepared blocks, f32, head-major so that a run of blocks is one contiguous run. Sequence number s with first row b begins at
// block b / 16 + s, which leaves every sequence room for a last block that is not full.
//   vec [heads][blocks][33][kd]             A_t q_t dim^-0.5 | R_s k_s | A_16; zero (A_16: one) past dim and for missing rows
//   v   [heads][col blocks][blocks][16][64] zero past vdim and for missing rows
//   p   [heads][blocks][16][16]             P_ts at [s][t], zero where s > t
//   o   [rows][heads * vdim]                outputs of the scan
//   u   [segments][heads][dim][vdim]        what a segment adds to the state; then the state at its start
//   keep [segments][heads][kd]              product of its decays
constexpr int kVecs = 2 * kBlock + 1;
struct Prepared {
  float *vec, *v, *p, *o, *u, *keep;
  int kd, cols, blocks, seg_len, segs;      // seg_len 0: sequences are not cut
  __device__ __forceinline__ float* vec_at(int h, int blk) const { return vec + (static_cast<int64_t>(h) * blocks + blk) * kVecs * kd; }
  __device__ __forceinline__ float* v_at(int h, int col, int blk) const { return v + ((static_cast<int64_t>(h) * cols + col) * blocks + blk) * kBlock * kCols; }
  __device__ __forceinline__ float* p_at(int h, int blk) const { return p + (static_cast<int64_t>(h) * blocks + blk) * kBlock * kBlock; }
};
__device__ __forceinline__ int first_block(int begin, int seq) { return begin / kBlock + seq; }
int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
int col_blocks(int vdim) { return (vdim + kCols - 1) / kCols; }
// Rows of a segment, or 0: sequences stay whole. `kPerSm` CTAs of the scan fit an SM, where `kTime` is the time of a fixed amount
// of work by one, two or three of them; cutting costs another half of the work for the first pass.
int segment_rows(int heads, int vdim, int rows, int seqs) {
  constexpr int kPerSm = 3;
  constexpr double kTime[kPerSm + 1] = {0.0, 1.0, 0.6, 0.5};
  if (seqs < 1) return 0;
  const int64_t ctas = static_cast<int64_t>(col_blocks(vdim)) * heads * seqs;
  int best = 1;
  double best_time = 1e30;
  for (int n = 1; n <= 16 && (n == 1 || (rows / seqs >= 128 * n && ctas * n <= kPerSm * kNumSMs)); ++n) {
    const int64_t per_sm = (ctas * n + kNumSMs - 1) / kNumSMs, waves = (per_sm + kPerSm - 1) / kPerSm;
    const int64_t at_once = per_sm < kPerSm ? per_sm : kPerSm;
    const double time = static_cast<double>(waves * at_once) * kTime[at_once] / n * (n > 1 ? 1.5 : 1.0);
    if (time < 0.9 * best_time) {
      best_time = time;
      best = n;
    }
  }
  if (best == 1) return 0;
  return ((rows / seqs + best - 1) / best + kBlock - 1) / kBlock * kBlock;
}
// Lays the scratch out; `total` receives its floats.
Prepared prepared_of(float* scratch, int heads, int dim, int vdim, int rows, int all_seqs, int seqs, int64_t& total) {
  Prepared p;
  p.kd = padded_dim(dim);
  p.cols = col_blocks(vdim);
  p.blocks = rows / kBlock + all_seqs + 1;
  p.seg_len = segment_rows(heads, vdim, rows, seqs);
  p.segs = p.seg_len > 0 ? seqs + rows / p.seg_len : seqs;
  total = 0;
  const auto take = [&](int64_t n) {
    float* at = scratch + total;
    total += (n + 31) / 32 * 32;
    return at;
  };
  const int64_t hb = static_cast<int64_t>(heads) * p.blocks, cut = p.seg_len > 0 ? static_cast<int64_t>(p.segs) * heads : 0;
  p.vec = take(hb * kVecs * p.kd);
  p.v = take(hb * p.cols * kBlock * kCols);
  p.p = take(hb * kBlock * kBlock);
  p.o = take(static_cast<int64_t>(rows) * heads * vdim);
  p.u = take(cut * dim * vdim);
  p.keep = take(cut * p.kd);
  return p;
}

// 16 sums over a warp: lane l receives the one of x[l >> 1].
__device__ __forceinline__ float warp_sum16(const float (&x)[16], int lane) {
  float a[8], b[4], c[2];
  const bool h4 = lane & 16, h3 = lane & 8, h2 = lane & 4, h1 = lane & 2;
#pragma unroll
  for (int j = 0; j < 8; ++j) a[j] = (h4 ? x[8 + j] : x[j]) + __shfl_xor_sync(0xffffffffu, h4 ? x[j] : x[8 + j], 16);
#pragma unroll
  for (int j = 0; j < 4; ++j) b[j] = (h3 ? a[4 + j] : a[j]) + __shfl_xor_sync(0xffffffffu, h3 ? a[j] : a[4 + j], 8);
#pragma unroll
  for (int j = 0; j < 2; ++j) c[j] = (h2 ? b[2 + j] : b[j]) + __shfl_xor_sync(0xffffffffu, h2 ? b[j] : b[2 + j], 4);
  const float s = (h1 ? c[1] : c[0]) + __shfl_xor_sync(0xffffffffu, h1 ? c[0] : c[1], 2);
  return s + __shfl_xor_sync(0xffffffffu, s, 1);
}

// CTA = (block, head), a thread per VEC key channels. PAIR: two channels of a row are one aligned access.
template <typename T, int KD, bool PAIR>
__global__ void __launch_bounds__(KD == 32 ? 32 : KD / 2, 1024 / KD) gated_prep_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, const Prepared out, int first,
                                                                          int n_seqs, Status* status) {
  ptx::grid_dep_sync();
  constexpr int VEC = KD == 32 ? 1 : 2, kThreads = KD / VEC, kAccess = PAIR ? VEC : 1;
  __shared__ float part[kThreads / 32][kBlock * kBlock];
  int i = blockIdx.x;
  const int seq = find_tile(sq, first, first + n_seqs, kBlock, i), h = blockIdx.y, c = threadIdx.x * VEC, lane = threadIdx.x & 31;
  const int d = a.dim, e = a.vdim, nk = a.heads * d;
  if (seq < 0) return;      // uniform per CTA, as the return below
  ConvRow cr;
  const int row0 = sq.seq_rows[2 * seq] + i * kBlock;
  if (!cr.load(sq, seq, row0, sq.banks, status)) return;
  const int m = min(kBlock, cr.end - row0), blk = first_block(cr.begin, seq) + i;
  const T* src = static_cast<const T*>(a.proj) + row0 * a.ld + h * d + c;
  const float* zs = a.z + row0 * a.ld_z + h * d + c;
  const T* vs = static_cast<const T*>(a.proj) + row0 * a.ld + 2 * nk + h * e;
  // everything this block needs is requested before the first value is used; VEC divides kCols
  constexpr int N = VEC / kAccess;
  RawVec<T, kAccess> raw_q[kBlock][N], raw_k[kBlock][N], raw_v[kBlock][N];
  float q[kBlock][VEC], k[kBlock][VEC], g[kBlock][VEC], bias[VEC];
  const auto request_v = [&](int col) {
#pragma unroll
    for (int t = 0; t < kBlock; ++t)
#pragma unroll
      for (int v = 0; v < N; ++v) {
        raw_v[t][v].zero();
        if (t < m && col + v * kAccess < e) raw_v[t][v].load(vs + t * a.ld + col + v * kAccess);
      }
  };
  const auto write_v = [&](int col) {
    float* dst = out.v_at(h, col / kCols, blk) + col % kCols;
#pragma unroll
    for (int t = 0; t < kBlock; ++t) {
      float x[VEC];
#pragma unroll
      for (int v = 0; v < VEC; ++v) x[v] = raw_v[t][v / kAccess].get(v % kAccess);
      store_f32<VEC>(dst + t * kCols, x);
    }
  };
  request_v(c);
#pragma unroll
  for (int t = 0; t < kBlock; ++t)
#pragma unroll
    for (int v = 0; v < N; ++v) {
      float z[kAccess] = {};
      raw_q[t][v].zero();
      raw_k[t][v].zero();
      if (c + v * kAccess < d && t < m) {
        raw_q[t][v].load(src + t * a.ld + v * kAccess);
        raw_k[t][v].load(src + nk + t * a.ld + v * kAccess);
        load_f32<kAccess>(zs + t * a.ld_z + v * kAccess, z);
      }
#pragma unroll
      for (int j = 0; j < kAccess; ++j) g[t][v * kAccess + j] = z[j];
    }
#pragma unroll
  for (int v = 0; v < VEC; ++v) bias[v] = c + v < d ? a.decay_bias[h * d + c + v] : 0.0f;
  if (c < out.cols * kCols) write_v(c);
  for (int col = c + KD; col < out.cols * kCols; col += KD) {
    request_v(col);
    write_v(col);
  }
  const float q_scale = rsqrtf(static_cast<float>(d));
#pragma unroll
  for (int t = 0; t < kBlock; ++t)
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
      g[t][v] = c + v < d && t < m ? decay_of(g[t][v] + bias[v], a.inv_tau) : 1.0f;
      q[t][v] = raw_q[t][v / kAccess].get(v % kAccess) * q_scale;
      k[t][v] = raw_k[t][v / kAccess].get(v % kAccess);
    }
  float* vec = out.vec_at(h, blk) + c;
  float run[VEC], x[VEC];
#pragma unroll
  for (int v = 0; v < VEC; ++v) run[v] = 1.0f;
#pragma unroll
  for (int t = 0; t < kBlock; ++t) {
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
      run[v] *= g[t][v];
      x[v] = q[t][v] * run[v];
    }
    store_f32<VEC>(vec + t * KD, x);
  }
  store_f32<VEC>(vec + 2 * kBlock * KD, run);
#pragma unroll
  for (int v = 0; v < VEC; ++v) run[v] = 1.0f;
#pragma unroll
  for (int s = kBlock - 1; s >= 0; --s) {
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
      x[v] = k[s][v] * run[v];
      run[v] *= g[s][v];
    }
    store_f32<VEC>(vec + (kBlock + s) * KD, x);
  }
  float* mine = part[threadIdx.x >> 5];
#pragma unroll
  for (int s = 0; s < kBlock; ++s) {
    float pr[kBlock];
#pragma unroll
    for (int t = 0; t < kBlock; ++t) {
      pr[t] = 0.0f;
      if (t < s) continue;
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        if (t > s) k[s][v] *= g[t][v];
        pr[t] = fmaf(q[t][v], k[s][v], pr[t]);
      }
    }
    const float sum = warp_sum16(pr, lane);
    if ((lane & 1) == 0) mine[s * kBlock + (lane >> 1)] = sum;
  }
  __syncthreads();
  float* p = out.p_at(h, blk);
  for (int j = threadIdx.x; j < kBlock * kBlock; j += kThreads) {
    float s = 0.0f;
#pragma unroll
    for (int w = 0; w < kThreads / 32; ++w) s += part[w][j];
    p[j] = s;
  }
}

// P: pairs of key rows a lane holds; eight lanes hold a column.
template <int P>
struct ScanLayout {
  static constexpr int kD = 16 * P;
  static constexpr int kVec = kVecs * kD, kV = kBlock * kCols, kStage = kVec + kV;      // floats of one block
  static constexpr int kBytes = kStages * kStage * 4 + kStages * 8;
};

// Whole: a sequence from its state to its state. Local: a segment, from zero, to what it adds; no outputs, and nothing for a
// sequence's last segment. Segment: from the start state `carry` left, outputs; the last one leaves the sequence's state.
enum class Scan { kWhole, kLocal, kSegment };

// Lane (rg = lane & 7, quarter = lane >> 3) of warp w: value columns blk * 64 + 16 w + 4 quarter + 0..3, key rows by pair_row.
template <int P, Scan MODE>
__global__ void __launch_bounds__(128) gated_scan_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, const Prepared in, int first, int n_seqs, Status* status) {
  ptx::grid_dep_sync();
  using L = ScanLayout<P>;
  extern __shared__ __align__(128) float scan_sm[];
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int seg = blockIdx.z;
  const int seq = MODE == Scan::kWhole ? first + seg : find_tile(sq, first, first + n_seqs, in.seg_len, seg);
  if (seq < 0) return;      // uniform per CTA, as the returns below
  const int seq_begin = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (sq.seq_rows[2 * seq + 1] <= seq_begin || !cr.load(sq, seq, seq_begin, sq.banks, status)) return;
  int begin = seq_begin, n = cr.end - cr.begin;
  if constexpr (MODE != Scan::kWhole) {
    begin += seg * in.seg_len;
    n = min(in.seg_len, cr.end - begin);
  }
  const bool last = begin + n == cr.end;
  if (MODE == Scan::kLocal && last) return;
  const int d = a.dim, e = a.vdim, n_blocks = (n + kBlock - 1) / kBlock, block0 = first_block(seq_begin, seq) + (begin - seq_begin) / kBlock;
  const uint32_t bars = ptx::smem_u32(scan_sm + kStages * L::kStage);
  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) ptx::mbar_init(bars + 8 * s, 1);
    ptx::fence_mbar_init();
  }
  __syncthreads();
  const float *g_vec = in.vec_at(h, block0), *g_v = in.v_at(h, blockIdx.x, block0);
  const auto issue = [&](int i) {      // thread 0: start the copies of block i
    const uint32_t st = ptx::smem_u32(scan_sm + (i % kStages) * L::kStage), bar = bars + 8 * (i % kStages);
    ptx::mbar_arrive_expect_tx(bar, L::kStage * 4);
    ptx::bulk_load(st, g_vec + static_cast<int64_t>(i) * L::kVec, L::kVec * 4, bar);
    ptx::bulk_load(st + L::kVec * 4, g_v + static_cast<int64_t>(i) * L::kV, L::kV * 4, bar);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < kStages - 1 && i < n_blocks; ++i) issue(i);

  constexpr int RG = 8;
  const int rg = lane & 7, c4 = 16 * warp + 4 * (lane >> 3), col = blockIdx.x * kCols + c4;
  const bool b2 = lane & 4, b1 = lane & 2, b0 = lane & 1;
  const bool busy = blockIdx.x * kCols + 16 * warp < e;      // else the warp has no columns
  float* state = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e + col;
  float* u = in.u + (static_cast<int64_t>(blockIdx.z) * a.heads + h) * d * e + col;
  uint64_t S[P][4], kept[MODE == Scan::kLocal ? P : 1];
  load_state<P, 4, RG>(MODE == Scan::kSegment ? u : state, MODE == Scan::kLocal || (MODE == Scan::kWhole && cr.rd < 0), d, e, col, rg, S);
  if constexpr (MODE == Scan::kLocal) {
#pragma unroll
    for (int p = 0; p < P; ++p) kept[p] = pack2(1.0f, 1.0f);
  }
  // after the reduction of two rows a lane holds the output of row (lane >> 2) & 1, column lane & 3
  const int64_t o_ld = static_cast<int64_t>(a.heads) * e;
  const int my_row = (lane >> 2) & 1;
  float* o_dst = in.o + static_cast<int64_t>(begin + my_row) * o_ld + static_cast<int64_t>(h) * e + col + (lane & 3);
  const bool writes = col + (lane & 3) < e;
  bool failed = false;
  for (int i = 0; i < n_blocks; ++i) {
    // the stage of block i - 1 was released by the barrier at the end of that block
    if (threadIdx.x == 0 && i + kStages - 1 < n_blocks) issue(i + kStages - 1);
    if (!ptx::mbar_wait(bars + 8 * (i % kStages), (i / kStages) & 1)) {
      status_record(status, kTimeout, kSiteAttn, seq, i);
      failed = true;
    }
    const float* st = scan_sm + (i % kStages) * L::kStage;
    const int m = min(kBlock, n - i * kBlock);
    if (busy) {
      if constexpr (MODE != Scan::kLocal) {
#pragma unroll 2
        for (int t = 0; t < m; t += 2) {      // the block's rows past the sequence's end are zero
          uint64_t acc[2][4];
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            uint64_t q[P];
            load_pairs<P, RG>(st + (t + r) * L::kD, rg, q);
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[r][c] = mul2(S[0][c], q[0]);
#pragma unroll
            for (int p = 1; p < P; ++p)
#pragma unroll
              for (int c = 0; c < 4; ++c) acc[r][c] = fma2(S[p][c], q[p], acc[r][c]);
          }
          float x4[4], x2[2];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float r0 = half_sum(acc[0][c]), r1 = half_sum(acc[1][c]);
            x4[c] = (b2 ? r1 : r0) + __shfl_xor_sync(0xffffffffu, b2 ? r0 : r1, 4);
          }
#pragma unroll
          for (int j = 0; j < 2; ++j) x2[j] = (b1 ? x4[2 + j] : x4[j]) + __shfl_xor_sync(0xffffffffu, b1 ? x4[j] : x4[2 + j], 2);
          const float o = (b0 ? x2[1] : x2[0]) + __shfl_xor_sync(0xffffffffu, b0 ? x2[0] : x2[1], 1);
          if (writes && t + my_row < m) o_dst[static_cast<int64_t>(i * kBlock + t) * o_ld] = o;
        }
      }
      uint64_t g[P];
      load_pairs<P, RG>(st + 2 * kBlock * L::kD, rg, g);
#pragma unroll
      for (int p = 0; p < P; ++p) {
#pragma unroll
        for (int c = 0; c < 4; ++c) S[p][c] = mul2(S[p][c], g[p]);
        if constexpr (MODE == Scan::kLocal) kept[p] = mul2(kept[p], g[p]);
      }
#pragma unroll 4
      for (int t = 0; t < m; ++t) {
        const float4 v = *reinterpret_cast<const float4*>(st + L::kVec + t * kCols + c4);
        const uint64_t vv[4] = {pack2(v.x, v.x), pack2(v.y, v.y), pack2(v.z, v.z), pack2(v.w, v.w)};
        uint64_t k[P];
        load_pairs<P, RG>(st + (kBlock + t) * L::kD, rg, k);
#pragma unroll
        for (int p = 0; p < P; ++p)
#pragma unroll
          for (int c = 0; c < 4; ++c) S[p][c] = fma2(k[p], vv[c], S[p][c]);
      }
    }
    if (__syncthreads_or(failed)) break;      // also releases the stage
  }
  if (failed) {
    // let copies in flight land before the CTA's shared memory is released
    for (int s = 0; s < kStages; ++s) ptx::mbar_wait(bars + 8 * s, 0, 20000000ull) || ptx::mbar_wait(bars + 8 * s, 1, 20000000ull);
    return;
  }
  if constexpr (MODE == Scan::kLocal) {
    store_state<P, 4, RG>(u, d, e, col, rg, S);
    if (blockIdx.x == 0 && warp == 0 && lane < RG) {
      float* keep = in.keep + (static_cast<int64_t>(blockIdx.z) * a.heads + h) * L::kD;
#pragma unroll
      for (int p = 0; p < P; ++p) *reinterpret_cast<uint64_t*>(keep + pair_row<P, RG>(p, rg)) = kept[p];
    }
  } else if (MODE == Scan::kWhole || last) {
    store_state<P, 4, RG>(state, d, e, col, rg, S);
  }
}

// The state at the start of every segment of a sequence, in place of what the segment adds. One thread per state element.
__global__ void __launch_bounds__(256) gated_carry_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, const Prepared in, int first, Status* status) {
  ptx::grid_dep_sync();
  const int h = blockIdx.y, seq = first + blockIdx.z, size = a.dim * a.vdim, i = blockIdx.x * blockDim.x + threadIdx.x;
  const int begin = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (i >= size || sq.seq_rows[2 * seq + 1] <= begin || !cr.load(sq, seq, begin, sq.banks, status)) return;
  int seg0 = 0;
  for (int s = first; s < seq; ++s) seg0 += (max(0, sq.seq_rows[2 * s + 1] - sq.seq_rows[2 * s]) + in.seg_len - 1) / in.seg_len;
  const int n = (cr.end - begin + in.seg_len - 1) / in.seg_len, key = i / a.vdim;
  float S = cr.rd >= 0 ? a.state[(static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * size + i] : 0.0f;
  for (int j0 = 0; j0 < n; j0 += 8) {
    float add[8], keep[8];      // up to eight segments are requested before the first is used
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int64_t at = static_cast<int64_t>(seg0 + j0 + j) * a.heads + h;
      const bool more = j0 + j + 1 < n;
      add[j] = more ? in.u[at * size + i] : 0.0f;
      keep[j] = more ? in.keep[at * in.kd + key] : 0.0f;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (j0 + j < n) {
        in.u[(static_cast<int64_t>(seg0 + j0 + j) * a.heads + h) * size + i] = S;
        S = fmaf(keep[j], S, add[j]);
      }
  }
}

// o_t = scan's part + sum_{s <= t} P_ts v_s, then out = rms_norm(o) * w * silu(gate) * out_scale. CTA = (block, head), a warp takes
// four of the rows.
template <typename T, int VEC, int NJ>
__global__ void __launch_bounds__(128) gated_out_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, const Prepared in, int first, int n_seqs, Status* status) {
  ptx::grid_dep_sync();
  int blk = blockIdx.x;
  const int seq = find_tile(sq, first, first + n_seqs, kBlock, blk), h = blockIdx.y, lane = threadIdx.x & 31, e = a.vdim, t0 = (threadIdx.x >> 5) * 4;
  if (seq < 0) return;
  ConvRow cr;
  const int row0 = sq.seq_rows[2 * seq] + blk * kBlock;
  if (!cr.load(sq, seq, row0, sq.banks, status)) return;
  const int n = min(4, cr.end - row0 - t0);      // this warp's rows
  if (n <= 0) return;
  // lane s holds P_ts of the four rows
  float4 p = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  if (lane < kBlock) p = *reinterpret_cast<const float4*>(in.p_at(h, first_block(cr.begin, seq) + blk) + lane * kBlock + t0);
  const T* vs = static_cast<const T*>(a.proj) + row0 * a.ld + 2 * a.heads * a.dim + h * e;
  const T* gate = vs + t0 * a.ld + a.heads * e;
  const float* o = in.o + (static_cast<int64_t>(row0 + t0) * a.heads + h) * e;
  float v[4][NJ][VEC], ss[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
    RawVec<T, VEC> x[kBlock];
#pragma unroll
    for (int s = 0; s < kBlock; ++s) {
      x[s].zero();
      if (s < t0 + n && c < e) x[s].load(vs + s * a.ld + c);
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[r][j][i] = 0.0f;
      if (r < n && c < e) load_f32<VEC>(o + static_cast<int64_t>(r) * a.heads * e + c, v[r][j]);
    }
#pragma unroll
    for (int s = 0; s < kBlock; ++s) {      // P is zero for rows behind t
      const float ps[4] = {__shfl_sync(0xffffffffu, p.x, s), __shfl_sync(0xffffffffu, p.y, s), __shfl_sync(0xffffffffu, p.z, s), __shfl_sync(0xffffffffu, p.w, s)};
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float f = x[s].get(i);
#pragma unroll
        for (int r = 0; r < 4; ++r) v[r][j][i] = fmaf(ps[r], f, v[r][j][i]);
      }
    }
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss[r] = fmaf(v[r][j][i], v[r][j][i], ss[r]);
  }
  RawVec<T, VEC> z[4][NJ];
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      z[r][j].zero();
      if (r < n && (lane + 32 * j) * VEC < e) z[r][j].load(gate + r * a.ld + (lane + 32 * j) * VEC);
    }
  warp_sum4(ss);
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
    if (c >= e) continue;
    float w[VEC];
    load_f32<VEC>(a.norm_w + c, w);
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      if (r >= n) break;      // uniform
      const float f = a.out_scale / sqrtf(ss[r] / static_cast<float>(e) + a.eps);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[r][j][i] = v[r][j][i] * f * w[i] * ptx::silu(z[r][j].get(i));
      store_f32<VEC>(static_cast<T*>(a.out) + (row0 + t0 + r) * a.ld_out + static_cast<int64_t>(h) * e + c, v[r][j]);
    }
  }
}

// Thread (rg, cg): value columns [cg * VEC, + VEC), key rows rg + i * n_rg, eight of them in flight at a time.
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreadsDecode) gated_decode_kernel(const B2GatedLinearArgs a, const B2SeqRows sq, int n_cg, int n_rg, Status* status) {
  ptx::grid_dep_sync();
  __shared__ __align__(16) float red[kThreadsDecode * VEC];
  enum { kA = 0, kK = 1, kQ = 2 };
  __shared__ float vec[3][kMaxDim], scratch[33];
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

template <int P, Scan MODE>
int launch_scan_mode(const B2GatedLinearArgs& a, const B2SeqRows& s, const Prepared& p, int first, int n, Status* status, cudaStream_t stream) {
  using L = ScanLayout<P>;
  static DeviceOnce attr_once;
  if (const int rc = attr_once.max_smem(gated_scan_kernel<P, MODE>, L::kBytes)) return rc;
  launch_pdl(gated_scan_kernel<P, MODE>, dim3(p.cols, a.heads, p.segs), dim3(128), L::kBytes, stream, a, s, p, first, n, status);
  return last_launch_rc();
}
// Preparation and scan for key sizes up to KD.
template <typename T, int KD>
int launch_blocks(const B2GatedLinearArgs& a, const B2SeqRows& s, const Prepared& p, int first, int n, bool pair, Status* status, cudaStream_t stream) {
  constexpr int P = KD / 16;
  auto prep = pair ? gated_prep_kernel<T, KD, true> : gated_prep_kernel<T, KD, false>;
  launch_pdl(prep, dim3(s.rows / kBlock + n, a.heads), dim3(KD == 32 ? 32 : KD / 2), 0, stream, a, s, p, first, n, status);
  if (const int rc = last_launch_rc()) return rc;
  if (p.seg_len == 0) return launch_scan_mode<P, Scan::kWhole>(a, s, p, first, n, status, stream);
  if (const int rc = launch_scan_mode<P, Scan::kLocal>(a, s, p, first, n, status, stream)) return rc;
  launch_pdl(gated_carry_kernel, dim3((a.dim * a.vdim + 255) / 256, a.heads, n), dim3(256), 0, stream, a, s, p, first, status);
  if (const int rc = last_launch_rc()) return rc;
  return launch_scan_mode<P, Scan::kSegment>(a, s, p, first, n, status, stream);
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
  // two channels at a time: every head, row and block begins at an even element, z and the projection at an aligned address
  const bool pair = a.dim % 2 == 0 && a.vdim % 2 == 0 && a.ld % 2 == 0 && a.ld_z % 2 == 0 && reinterpret_cast<uintptr_t>(a.proj) % (2 * sizeof(T)) == 0 &&
                    reinterpret_cast<uintptr_t>(a.z) % 8 == 0;
  const dim3 grid(s.rows / kBlock + n_prefill, a.heads);
  int64_t total;
  const Prepared p = prepared_of(a.scratch, a.heads, a.dim, a.vdim, s.rows, s.seqs, n_prefill, total);
  int rc;
  switch (p.kd) {
    case 32: rc = launch_blocks<T, 32>(a, s, p, first, n_prefill, pair, status, stream); break;
    case 64: rc = launch_blocks<T, 64>(a, s, p, first, n_prefill, pair, status, stream); break;
    case 128: rc = launch_blocks<T, 128>(a, s, p, first, n_prefill, pair, status, stream); break;
    default: rc = launch_blocks<T, 256>(a, s, p, first, n_prefill, pair, status, stream);
  }
  if (rc) return rc;
  if (v4 && a.vdim <= 128) launch_pdl(gated_out_kernel<T, 4, 1>, grid, dim3(128), 0, stream, a, s, p, first, n_prefill, status);
  else if (v4) launch_pdl(gated_out_kernel<T, 4, 2>, grid, dim3(128), 0, stream, a, s, p, first, n_prefill, status);
  else launch_pdl(gated_out_kernel<T, 1, 8>, grid, dim3(128), 0, stream, a, s, p, first, n_prefill, status);
  return last_launch_rc();
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int64_t b2_gated_linear_scratch_floats(int heads, int dim, int vdim, int rows, int all_seqs, int seqs) {
  int64_t total;
  prepared_of(nullptr, heads, dim, vdim, rows, all_seqs, seqs, total);
  return total;
}
// Kernels that one call launches for its prompt chunks.
extern "C" int b2_gated_linear_prefill_launches(int heads, int vdim, int rows, int seqs) { return segment_rows(heads, vdim, rows, seqs) > 0 ? 5 : 3; }

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
