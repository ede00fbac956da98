// Gated delta rule with one decay per key channel, or one per head. State S [dim, vdim] per head, all of it in f32:
//   S <- g * S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q
// Three kernels:
//   prep    every row and head at once: short convolution and silu of q, k, v, unit norms, decays, step sizes, and the few
//           dot products of neighbouring rows that the scan needs; f32, laid out the way the other two read them
//   decode  one row per sequence. CTA = (head, sequence): S streams through registers once, output norm and gate fused
//   scan    any number of rows. CTA = (32 value columns, head, sequence): S stays in the registers of four warps, which walk
//           over the rows two at a time while bulk copies bring the next rows into shared memory; norm and gate follow in a
//           kernel of their own
// Rows go in pairs, because a pair costs one reduction over the key rows instead of two. With S the state before the pair,
//   S^T k of row 1 = S . (g1 k1)                 of row 2 = S . (g1 g2 k2) + u1 ((g2 k1) . k2)      (likewise for q)
//   S after        = g1 g2 S + (g2 k1) u1^T + k2 u2^T
// so the prepared vectors g1 k1, g1 q1, g1 g2 k2, g1 g2 q2, g1 g2, g2 k1, k2 and a few scalars are all a pair needs.
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/recurrence.cuh"
#include "b2/short_conv.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kMaxDim = 256;
constexpr float kUnitEps = 1e-6f;
constexpr int kTile = 8;         // pairs of one shared-memory stage of the scan
constexpr int kStages = 3;
constexpr int kCols = 32;        // value columns of a scan CTA

__device__ __forceinline__ float sigmoid(float x) { return ptx::rcp(1.0f + ptx::ex2(-x * ptx::kLog2e)); }
__device__ __forceinline__ float gate_value(const B2DeltaArgs& a, float z) { return a.gate_silu ? z * sigmoid(z) : sigmoid(z); }
// The gates of a head in a row.
template <typename T>
__device__ __forceinline__ const T* gate_row(const B2DeltaArgs& a, int row, int h) { return static_cast<const T*>(a.gate) + static_cast<int64_t>(row) * a.ld_gate + h * a.vdim; }

// Prepared pairs, f32, head-major so that a run of pairs is one contiguous block. Sequence number s with first row b starts at
// pair (b + s) / 2, which leaves every sequence room for a last pair that is half empty.
//   vec [heads][pairs][7][kd]            the vectors named above; zero (factors of S: one) past dim and for a missing row 2
//   v   [heads][col blocks][pairs][2][32]
//   sc  [heads][pairs][8]                beta1, k1 . q1, beta2, k2 . q2, (g2 k1) . k2, (g2 k1) . q2, -, -
enum PairVec { kGK1 = 0, kGQ1 = 1, kGK2 = 2, kGQ2 = 3, kGG = 4, kW1 = 5, kW2 = 6, kVecs = 7 };
struct Prepared {
  float* vec;
  float* v;
  float* sc;
  int kd, blocks, pairs;
  __device__ __forceinline__ float* vec_at(int h, int pair) const { return vec + (static_cast<int64_t>(h) * pairs + pair) * kVecs * kd; }
  __device__ __forceinline__ float* v_at(int h, int blk, int pair) const { return v + ((static_cast<int64_t>(h) * blocks + blk) * pairs + pair) * 2 * kCols; }
  __device__ __forceinline__ float* sc_at(int h, int pair) const { return sc + (static_cast<int64_t>(h) * pairs + pair) * 8; }
};
__device__ __forceinline__ int first_pair(int begin, int seq) { return (begin + seq) >> 1; }

int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
int pair_count(int rows, int seqs) { return (rows + seqs) / 2 + 1; }
int64_t scratch_floats(int heads, int dim, int vdim, int rows, int seqs) {
  const int64_t blocks = (vdim + kCols - 1) / kCols;
  return static_cast<int64_t>(pair_count(rows, seqs)) * heads * (kVecs * padded_dim(dim) + blocks * 2 * kCols + 8);
}
Prepared prepared_of(const B2DeltaArgs& a, const B2SeqRows& s) {
  Prepared p;
  p.kd = padded_dim(a.dim);
  p.blocks = (a.vdim + kCols - 1) / kCols;
  p.pairs = pair_count(s.rows, s.seqs);
  p.vec = a.scratch;
  p.v = p.vec + static_cast<int64_t>(p.pairs) * a.heads * kVecs * p.kd;
  p.sc = p.v + static_cast<int64_t>(p.pairs) * a.heads * p.blocks * 2 * kCols;
  return p;
}

// ------------------------------------------------------------------------------------------------------------
// prep
// ------------------------------------------------------------------------------------------------------------
// Warp = (TT consecutive rows of one sequence, head); tiles count from each sequence's first row, so a pair of rows never
// straddles two warps. Lane l holds channels (l + 32 j) * VEC.
template <typename T, int VEC, int NJ, int TAPS, int TT>
__global__ void __launch_bounds__(128, TAPS > 0 && NJ == 1 ? 6 : 1) delta_prep_kernel(const B2DeltaArgs a, const B2SeqRows sq, const Prepared out, Status* status) {
  ptx::grid_dep_sync();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * 4 + warp;
  if (h >= a.heads) return;
  int tile = static_cast<int>(blockIdx.x);
  const int seq = find_tile(sq, 0, sq.seqs, TT, tile);
  if (seq < 0) return;
  const int row0 = sq.seq_rows[2 * seq] + tile * TT;
  ConvRow cr;
  if (!cr.load(sq, seq, row0, sq.banks, status)) return;
  const int n = min(TT, cr.end - row0);
  const int d = a.dim, e = a.vdim, per = a.heads / a.kv_heads, kh = h / per, ck = a.kv_heads * d;
  const ConvSource<T> src{static_cast<const T*>(a.proj), a.ld, a.conv_w, static_cast<T*>(a.conv_state), a.taps, 2 * ck + a.heads * e, sq.banks};
  const bool save_qk = h % per == 0;

  float q[NJ][TT][VEC], k[NJ][TT][VEC], g[NJ][TT][VEC];
  const float rate = a.neg_rate[h] * ptx::kLog2e;
  float head_g[TT];      // one decay for all channels
  if (a.head_decay) {
    const float bias = a.dt_bias[h];
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      float z[1] = {0.0f};
      if (t < n) load_f32<1>(static_cast<const T*>(a.decay) + static_cast<int64_t>(row0 + t) * a.ld_decay + h, z);
      head_g[t] = ptx::ex2(rate * softplus_fast(z[0] + bias));
    }
  }
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
    if (c < d) {
      conv_rows<T, VEC, TAPS, TT>(src, cr, row0, n, kh * d + c, save_qk, q[j]);
      conv_rows<T, VEC, TAPS, TT>(src, cr, row0, n, ck + kh * d + c, save_qk, k[j]);
      float bias[VEC] = {};
      if (!a.head_decay) load_f32<VEC>(a.dt_bias + h * d + c, bias);
#pragma unroll
      for (int t = 0; t < TT; ++t) {
        float z[VEC] = {};
        if (t < n && !a.head_decay) load_f32<VEC>(static_cast<const T*>(a.decay) + static_cast<int64_t>(row0 + t) * a.ld_decay + h * d + c, z);
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          // a row that is not there changes nothing
          q[j][t][v] = t < n ? ptx::silu(q[j][t][v]) : 0.0f;
          k[j][t][v] = t < n ? ptx::silu(k[j][t][v]) : 0.0f;
          g[j][t][v] = t < n ? (a.head_decay ? head_g[t] : ptx::ex2(rate * softplus_fast(z[v] + bias[v]))) : 1.0f;
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
  float qq[TT], kk[TT], kq[TT];
#pragma unroll
  for (int t = 0; t < TT; ++t) {
    qq[t] = kk[t] = kq[t] = 0.0f;
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        qq[t] = fmaf(q[j][t][v], q[j][t][v], qq[t]);
        kk[t] = fmaf(k[j][t][v], k[j][t][v], kk[t]);
        kq[t] = fmaf(q[j][t][v], k[j][t][v], kq[t]);
      }
  }
  if constexpr (TT == 4) {
    warp_sum4(qq);
    warp_sum4(kk);
    warp_sum4(kq);
  } else {
#pragma unroll
    for (int t = 0; t < TT; ++t) {
      qq[t] = warp_sum(qq[t]);
      kk[t] = warp_sum(kk[t]);
      kq[t] = warp_sum(kq[t]);
    }
  }
#pragma unroll
  for (int t = 0; t < TT; ++t) {
    const float rq = q_scale * rsqrtf(qq[t] + kUnitEps), rk = rsqrtf(kk[t] + kUnitEps);
    kq[t] *= rq * rk;
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        q[j][t][v] *= rq;
        k[j][t][v] *= rk;
      }
  }
  const int pair0 = first_pair(cr.begin, seq) + (row0 - cr.begin) / 2;
#pragma unroll
  for (int t = 0; t < TT; t += 2) {
    if (t >= n) break;
    constexpr bool kTwo = TT > 1;
    float* dst = out.vec_at(h, pair0 + t / 2);
    float wk = 0.0f, wq = 0.0f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = (lane + 32 * j) * VEC;
      float x[kVecs][VEC];
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        const float g1 = g[j][t][v], k1 = k[j][t][v];
        x[kGK1][v] = g1 * k1;
        x[kGQ1][v] = g1 * q[j][t][v];
        if constexpr (kTwo) {
          const float g2 = g[j][t + 1][v], k2 = k[j][t + 1][v], q2 = q[j][t + 1][v], gg = g1 * g2, w1 = g2 * k1;
          x[kGK2][v] = gg * k2;
          x[kGQ2][v] = gg * q2;
          x[kGG][v] = gg;
          x[kW1][v] = w1;
          x[kW2][v] = k2;
          wk = fmaf(w1, k2, wk);
          wq = fmaf(w1, q2, wq);
        } else {
          x[kGK2][v] = x[kGQ2][v] = x[kW2][v] = 0.0f;
          x[kGG][v] = g1;
          x[kW1][v] = k1;
        }
      }
      if (c < out.kd) {
#pragma unroll
        for (int i = 0; i < kVecs; ++i) store_f32<VEC>(dst + i * out.kd + c, x[i]);
      }
    }
    if constexpr (kTwo) {
      wk = warp_sum(wk);
      wq = warp_sum(wq);
    }
    if (lane == 0) {
      const bool two = kTwo && t + 1 < n;
      float b1[1], b2v[1] = {0.0f};
      const T* b = static_cast<const T*>(a.proj) + static_cast<int64_t>(row0 + t) * a.ld + a.b_off + h;
      load_f32<1>(b, b1);
      if (two) load_f32<1>(b + a.ld, b2v);
      float* sc = out.sc_at(h, pair0 + t / 2);
      *reinterpret_cast<float4*>(sc) = make_float4(sigmoid(b1[0]), kq[t], two ? sigmoid(b2v[0]) : 0.0f, two ? kq[t + (kTwo ? 1 : 0)] : 0.0f);
      *reinterpret_cast<float4*>(sc + 4) = make_float4(wk, wq, 0.0f, 0.0f);
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
      if (t >= ((n + 1) & ~1)) break;
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[t][i] = t < n ? ptx::silu(v[t][i]) : 0.0f;
      store_f32<VEC>(out.v_at(h, c / kCols, pair0 + t / 2) + (t & 1) * kCols + c % kCols, v[t]);
    }
  }
}

template <typename T, int VEC, int NJ, int TAPS, int TT>
int launch_prep(const B2DeltaArgs& a, const B2SeqRows& s, bool one_row_each, Status* status, cudaStream_t stream) {
  const int tiles = one_row_each ? s.seqs : (s.rows + TT - 1) / TT + s.seqs;      // every sequence may end in a partial tile
  launch_pdl(delta_prep_kernel<T, VEC, NJ, TAPS, TT>, dim3(tiles, (a.heads + 3) / 4), dim3(128), 0, stream, a, s, prepared_of(a, s), status);
  return last_launch_rc();
}

// Whether rows of four elements can be read at once from every multiple of four on.
template <typename T>
bool vec4_rows(const void* p, int64_t ld) { return ld % 4 == 0 && reinterpret_cast<uintptr_t>(p) % (4 * sizeof(T)) == 0; }

template <typename T>
int dispatch_prep(const B2DeltaArgs& a, const B2SeqRows& s, bool one_row_each, Status* status, cudaStream_t stream) {
  const int m = a.dim > a.vdim ? a.dim : a.vdim;
  if (a.taps == 4 && a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ld % 4 == 0 && (a.head_decay || vec4_rows<T>(a.decay, a.ld_decay))) {
    if (m <= 128)
      return one_row_each ? launch_prep<T, 4, 1, 4, 1>(a, s, true, status, stream) : launch_prep<T, 4, 1, 4, 4>(a, s, false, status, stream);
    return launch_prep<T, 4, 2, 4, 2>(a, s, one_row_each, status, stream);
  }
  return launch_prep<T, 1, 8, 0, 2>(a, s, one_row_each, status, stream);
}

// ------------------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------------------
// Both forms: thread (rg, cg) handles columns [cg * VEC, + VEC) and key rows rg + i * n_rg. `finish` normalises, gates and
// writes the outputs that the threads with rg == 0 hold.
template <typename T, int VEC>
__device__ __forceinline__ void decode_finish(const B2DeltaArgs& a, int row, int h, int cg, bool owner, float (&o)[VEC], float* scratch) {
  float ss = 0.0f;
#pragma unroll
  for (int v = 0; v < VEC; ++v) ss = fmaf(o[v], o[v], ss);
  ss = block_sum(ss, scratch);
  if (!owner) return;
  const float r = rsqrtf(ss / static_cast<float>(a.vdim) + a.eps);
  float z[VEC], w[VEC];
  load_f32<VEC>(gate_row<T>(a, row, h) + cg * VEC, z);
  load_f32<VEC>(a.norm_w + cg * VEC, w);
#pragma unroll
  for (int v = 0; v < VEC; ++v) o[v] = o[v] * r * w[v] * gate_value(a, z[v]);
  store_f32<VEC>(static_cast<T*>(a.out) + static_cast<int64_t>(row) * a.ld_out + static_cast<int64_t>(h) * a.vdim + cg * VEC, o);
}

// Plain form for sizes the pipelined one does not take: one CTA per (head, sequence), S read twice.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) delta_decode_plain_kernel(const B2DeltaArgs a, const B2SeqRows sq, const Prepared in, int n_cg, int n_rg,
                                                                 Status* status) {
  ptx::grid_dep_sync();
  __shared__ __align__(16) float red[2][256 * VEC];
  __shared__ float scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, d = a.dim, e = a.vdim;
  ConvRow cr;
  const int row = decode_row(sq, seq, cr, status);
  if (row < 0) return;      // uniform per CTA
  const int cg = threadIdx.x % n_cg, rg = threadIdx.x / n_cg, pair = first_pair(cr.begin, seq);
  const bool active = rg < n_rg, fresh = cr.rd < 0;
  float* S = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e + cg * VEC;
  const float *vec = in.vec_at(h, pair), *sc = in.sc_at(h, pair);
  float ks[VEC] = {}, qs[VEC] = {}, o[VEC] = {};
  if (active) {
    for (int r = rg; r < d && !fresh; r += n_rg) {
      float x[VEC];
      load_f32<VEC>(S + static_cast<int64_t>(r) * e, x);
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        ks[v] = fmaf(x[v], vec[kGK1 * in.kd + r], ks[v]);
        qs[v] = fmaf(x[v], vec[kGQ1 * in.kd + r], qs[v]);
      }
    }
    store_f32<VEC>(red[0] + rg * e + cg * VEC, ks);
    store_f32<VEC>(red[1] + rg * e + cg * VEC, qs);
  }
  __syncthreads();
  if (active) {
    float u[VEC], sum[VEC] = {};
    load_f32<VEC>(in.v_at(h, cg * VEC / kCols, pair) + cg * VEC % kCols, u);
    for (int i = 0; i < n_rg; ++i) {
      load_f32<VEC>(red[0] + i * e + cg * VEC, ks);
#pragma unroll
      for (int v = 0; v < VEC; ++v) sum[v] += ks[v];
    }
#pragma unroll
    for (int v = 0; v < VEC; ++v) u[v] = sc[0] * (u[v] - sum[v]);
    for (int r = rg; r < d; r += n_rg) {
      float x[VEC] = {};
      if (!fresh) load_f32<VEC>(S + static_cast<int64_t>(r) * e, x);
#pragma unroll
      for (int v = 0; v < VEC; ++v) x[v] = fmaf(vec[kW1 * in.kd + r], u[v], x[v] * vec[kGG * in.kd + r]);
      store_f32<VEC>(S + static_cast<int64_t>(r) * e, x);
    }
    if (rg == 0) {
      for (int i = 0; i < n_rg; ++i) {
        load_f32<VEC>(red[1] + i * e + cg * VEC, qs);
#pragma unroll
        for (int v = 0; v < VEC; ++v) o[v] += qs[v];
      }
#pragma unroll
      for (int v = 0; v < VEC; ++v) o[v] = fmaf(u[v], sc[1], o[v]);
    }
  }
  decode_finish<T, VEC>(a, row, h, cg, rg == 0, o, scratch);
}

// Pipelined form: persistent CTAs walk over (sequence, head) items. A stage holds one item: S [d][e], then the row's seven
// vectors, values and scalars. While one item is computed in place, the next one's copies are on their way in and the
// previous one's state is on its way out.
constexpr int kDecodeThreads = 512;
struct DecodeLayout {
  int state, vec, v, sc, stage, stages, n_cg, n_rg, bytes;      // floats; `bytes`: dynamic shared memory
};
template <typename T>
__global__ void __launch_bounds__(kDecodeThreads, 2) delta_decode_kernel(const B2DeltaArgs a, const B2SeqRows sq, const Prepared in, const DecodeLayout L,
                                                                        int n_seqs, Status* status) {
  ptx::grid_dep_sync();
  extern __shared__ __align__(128) float dec_sm[];
  __shared__ float scratch[33];
  const int tid = threadIdx.x, d = a.dim, e = a.vdim, H = a.heads, total = n_seqs * H;
  float* red_k = dec_sm + L.stages * L.stage;
  float* red_q = red_k + L.n_rg * e;
  const uint32_t bars = ptx::smem_u32(red_q + L.n_rg * e);
  if (tid == 0) {
    for (int s = 0; s < L.stages; ++s) ptx::mbar_init(bars + 8 * s, 1);
    ptx::fence_mbar_init();
  }
  __syncthreads();
  const int cg = tid % L.n_cg, rg = tid / L.n_cg;
  const bool active = rg < L.n_rg;
  struct Item { int index, row, seq, h; ConvRow cr; };
  const auto find = [&](int i) {      // the first usable item at or after i of this CTA; the same in every thread
    Item it{};
    for (; i < total; i += gridDim.x) {
      it.seq = i / H;
      it.h = i % H;
      it.row = decode_row(sq, it.seq, it.cr, status);
      if (it.row >= 0) break;
    }
    it.index = i;
    return it;
  };
  const auto state_of = [&](const Item& it) { return a.state + (static_cast<int64_t>(it.cr.wr >> 1) * H + it.h) * d * e; };
  const auto issue = [&](const Item& it, int s) {      // thread 0
    float* st = dec_sm + s * L.stage;
    const uint32_t bar = bars + 8 * s;
    const int pair = first_pair(it.cr.begin, it.seq), state_bytes = it.cr.rd >= 0 ? d * e * 4 : 0;
    ptx::mbar_arrive_expect_tx(bar, static_cast<uint32_t>(state_bytes + kVecs * in.kd * 4 + in.blocks * kCols * 4 + 32));
    if (state_bytes) ptx::bulk_load(ptx::smem_u32(st), state_of(it), state_bytes, bar);
    ptx::bulk_load(ptx::smem_u32(st + L.vec), in.vec_at(it.h, pair), kVecs * in.kd * 4, bar);
    for (int b = 0; b < in.blocks; ++b) ptx::bulk_load(ptx::smem_u32(st + L.v + b * kCols), in.v_at(it.h, b, pair), kCols * 4, bar);
    ptx::bulk_load(ptx::smem_u32(st + L.sc), in.sc_at(it.h, pair), 32, bar);
  };
  Item cur = find(blockIdx.x);
  if (tid == 0 && cur.index < total) issue(cur, 0);
  bool failed = false;
  int k = 0;
  for (; cur.index < total; ++k) {
    const int s = k % L.stages;
    const Item nxt = find(cur.index + gridDim.x);
    if (tid == 0 && nxt.index < total) {
      // the stage's last state must have been read out: with three stages the newest store may still be pending
      if (L.stages >= 3) ptx::tma_store_wait_read<1>();
      else ptx::tma_store_wait_read<0>();
      issue(nxt, (k + 1) % L.stages);
    }
    if (!ptx::mbar_wait(bars + 8 * s, (k / L.stages) & 1)) {
      status_record(status, kTimeout, kSiteAttn, cur.seq, k);
      failed = true;
    }
    if (__syncthreads_or(failed)) break;
    float* st = dec_sm + s * L.stage + cg * 4;
    const float* vec = dec_sm + s * L.stage + L.vec;
    const float* sc = dec_sm + s * L.stage + L.sc;
    const bool fresh = cur.cr.rd < 0;
    float o[4] = {};
    if (active) {
      float ks[4] = {}, qs[4] = {};
      if (!fresh) {
#pragma unroll 4
        for (int r = rg; r < d; r += L.n_rg) {
          float x[4];
          load_f32<4>(st + r * e, x);
          const float gk = vec[kGK1 * in.kd + r], gq = vec[kGQ1 * in.kd + r];
#pragma unroll
          for (int v = 0; v < 4; ++v) {
            ks[v] = fmaf(x[v], gk, ks[v]);
            qs[v] = fmaf(x[v], gq, qs[v]);
          }
        }
      }
      store_f32<4>(red_k + rg * e + cg * 4, ks);
      store_f32<4>(red_q + rg * e + cg * 4, qs);
    }
    __syncthreads();
    if (active) {
      float u[4], sum[4] = {};
      load_f32<4>(dec_sm + s * L.stage + L.v + cg * 4, u);
      for (int i = 0; i < L.n_rg; ++i) {
        float x[4];
        load_f32<4>(red_k + i * e + cg * 4, x);
#pragma unroll
        for (int v = 0; v < 4; ++v) sum[v] += x[v];
      }
#pragma unroll
      for (int v = 0; v < 4; ++v) u[v] = sc[0] * (u[v] - sum[v]);
#pragma unroll 4
      for (int r = rg; r < d; r += L.n_rg) {
        float x[4] = {};
        if (!fresh) load_f32<4>(st + r * e, x);
        const float gg = vec[kGG * in.kd + r], w = vec[kW1 * in.kd + r];
#pragma unroll
        for (int v = 0; v < 4; ++v) x[v] = fmaf(w, u[v], x[v] * gg);
        store_f32<4>(st + r * e, x);
      }
      if (rg == 0) {
        for (int i = 0; i < L.n_rg; ++i) {
          float x[4];
          load_f32<4>(red_q + i * e + cg * 4, x);
#pragma unroll
          for (int v = 0; v < 4; ++v) o[v] += x[v];
        }
#pragma unroll
        for (int v = 0; v < 4; ++v) o[v] = fmaf(u[v], sc[1], o[v]);
      }
    }
    ptx::fence_proxy_async_smem();      // the new state, written by ordinary stores, is about to be copied out
    __syncthreads();
    if (tid == 0) {
      ptx::bulk_store(state_of(cur), ptx::smem_u32(dec_sm + s * L.stage), d * e * 4);
      ptx::tma_store_commit();
    }
    decode_finish<T, 4>(a, cur.row, cur.h, cg, rg == 0, o, scratch);
    cur = nxt;
  }
  if (tid == 0) {
    ptx::tma_store_wait<0>();
    if (failed)      // let copies in flight land before the CTA's shared memory is released
      for (int s = 0; s < L.stages; ++s) ptx::mbar_wait(bars + 8 * s, 0, 20000000ull) || ptx::mbar_wait(bars + 8 * s, 1, 20000000ull);
  }
}

template <typename T>
int dispatch_decode(const B2DeltaArgs& a, const B2SeqRows& s, int n, Status* status, cudaStream_t stream) {
  const bool v4 = a.vdim % 4 == 0 && vec4_rows<T>(a.gate, a.ld_gate) && a.ld_out % 4 == 0;
  const Prepared in = prepared_of(a, s);
  DecodeLayout L{};
  if (v4) {
    L.state = a.dim * a.vdim;
    L.vec = L.state;
    L.v = L.vec + kVecs * in.kd;
    L.sc = L.v + in.blocks * kCols;
    L.stage = (L.sc + 8 + 31) / 32 * 32;
    L.n_cg = a.vdim / 4;
    L.n_rg = kDecodeThreads / L.n_cg;
    if (L.n_rg > a.dim) L.n_rg = a.dim;
    for (L.stages = 3; L.stages >= 2; --L.stages) {
      L.bytes = (L.stages * L.stage + 2 * L.n_rg * a.vdim) * 4 + L.stages * 8;
      if (L.bytes <= kMaxSmemPerCta - 1024) break;
    }
  }
  if (L.stages >= 2) {
    static DeviceOnce attr_once;
    if (const int rc = attr_once.max_smem(delta_decode_kernel<T>, kMaxSmemPerCta - 1024)) return rc;
    int per_sm = kMaxSmemPerCta / (L.bytes + 1024);
    if (per_sm > 2) per_sm = 2;
    const int64_t items = static_cast<int64_t>(n) * a.heads;
    const int grid = static_cast<int>(items < static_cast<int64_t>(per_sm) * kNumSMs ? items : per_sm * kNumSMs);
    launch_pdl(delta_decode_kernel<T>, dim3(grid), dim3(kDecodeThreads), L.bytes, stream, a, s, in, L, n, status);
    return last_launch_rc();
  }
  const int n_cg = v4 ? a.vdim / 4 : a.vdim;
  int n_rg = 256 / n_cg;
  if (n_rg > a.dim) n_rg = a.dim;
  if (v4) launch_pdl(delta_decode_plain_kernel<T, 4>, dim3(a.heads, n), dim3(256), 0, stream, a, s, in, n_cg, n_rg, status);
  else launch_pdl(delta_decode_plain_kernel<T, 1>, dim3(a.heads, n), dim3(256), 0, stream, a, s, in, n_cg, n_rg, status);
  return last_launch_rc();
}

// ------------------------------------------------------------------------------------------------------------
// scan
// ------------------------------------------------------------------------------------------------------------
template <int P>
struct ScanLayout {
  static constexpr int kD = 32 * P;
  static constexpr int kVec = kVecs * kD, kV = 2 * kCols, kSc = 8;       // floats per pair
  static constexpr int kOffV = kTile * kVec, kOffSc = kOffV + kTile * kV;
  static constexpr int kStage = kOffSc + kTile * kSc;
  static constexpr int kBytes = kStages * kStage * 4 + kStages * 8;
};
// Lane (rg = lane & 15, half = lane >> 4) of warp w: value columns col0 + 8 w + 4 half + 0..3.
template <int P>
__global__ void __launch_bounds__(128) delta_scan_kernel(const B2DeltaArgs a, const B2SeqRows sq, const Prepared in, int first, Status* status) {
  ptx::grid_dep_sync();
  using L = ScanLayout<P>;
  extern __shared__ __align__(128) float scan_sm[];
  const int seq = first + blockIdx.z, h = blockIdx.y, blk = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int begin = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (sq.seq_rows[2 * seq + 1] <= begin || !cr.load(sq, seq, begin, sq.banks, status)) return;      // uniform per CTA
  const int d = a.dim, e = a.vdim, n = cr.end - cr.begin;
  const int n_pairs = (n + 1) >> 1, n_tiles = (n_pairs + kTile - 1) / kTile, pair0 = first_pair(begin, seq);
  const uint32_t bars = ptx::smem_u32(scan_sm + kStages * L::kStage);
  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) ptx::mbar_init(bars + 8 * s, 1);
    ptx::fence_mbar_init();
  }
  __syncthreads();
  const float *g_vec = in.vec_at(h, pair0), *g_v = in.v_at(h, blk, pair0), *g_sc = in.sc_at(h, pair0);
  const auto issue = [&](int i) {      // thread 0: start the copies of tile i
    const int m = min(kTile, n_pairs - i * kTile);
    const uint32_t st = ptx::smem_u32(scan_sm + (i % kStages) * L::kStage), bar = bars + 8 * (i % kStages);
    ptx::mbar_arrive_expect_tx(bar, static_cast<uint32_t>(m * (L::kVec + L::kV + L::kSc) * 4));
    ptx::bulk_load(st, g_vec + static_cast<int64_t>(i) * kTile * L::kVec, m * L::kVec * 4, bar);
    ptx::bulk_load(st + L::kOffV * 4, g_v + static_cast<int64_t>(i) * kTile * L::kV, m * L::kV * 4, bar);
    ptx::bulk_load(st + L::kOffSc * 4, g_sc + static_cast<int64_t>(i) * kTile * L::kSc, m * L::kSc * 4, bar);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < kStages - 1 && i < n_tiles; ++i) issue(i);

  const int rg = lane & 15, c4 = 8 * warp + 4 * (lane >> 4), col = blk * kCols + c4, half = lane & 16;
  // after the reduction over the 16 row groups a lane holds one sum: kind (S^T k, S^T q) = bit 3, row of the pair = bit 2,
  // column = bits 1, 0
  const bool is_q = lane & 8, second = lane & 4, b1 = lane & 2, b0 = lane & 1;
  const int mine = lane & 3;
  float* state = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.heads + h) * d * e + col;
  uint64_t S[P][4];
  load_state<P, 4>(state, cr.rd < 0, d, e, col, rg, S);
  const int64_t o_ld = static_cast<int64_t>(a.heads) * e;
  float* o_dst = a.o_raw + static_cast<int64_t>(begin + (second ? 1 : 0)) * o_ld + static_cast<int64_t>(h) * e + col + mine;
  const bool writes = is_q && col + mine < e;
  bool failed = false;
  for (int i = 0; i < n_tiles; ++i) {
    // the stage of tile i - 1 was released by the barrier at the end of that tile
    if (threadIdx.x == 0 && i + kStages - 1 < n_tiles) issue(i + kStages - 1);
    if (!ptx::mbar_wait(bars + 8 * (i % kStages), (i / kStages) & 1)) {
      status_record(status, kTimeout, kSiteAttn, seq, i);
      failed = true;
    }
    const float* st = scan_sm + (i % kStages) * L::kStage;
    const int m = min(kTile, n_pairs - i * kTile);
#pragma unroll 1
    for (int t = 0; t < m; ++t) {
      const float* vec = st + t * L::kVec;
      const float4 sc = *reinterpret_cast<const float4*>(st + L::kOffSc + t * L::kSc);              // beta1, k1.q1, beta2, k2.q2
      const float2 cross = *reinterpret_cast<const float2*>(st + L::kOffSc + t * L::kSc + 4);      // w1.k2, w1.q2
      const float* v = st + L::kOffV + t * L::kV + c4 + mine;
      const float v1 = v[0], v2 = v[kCols];
      uint64_t acc[4][4];      // S^T of g1 k1, g1 g2 k2, g1 q1, g1 g2 q2; even and odd rows apart
      const int which[4] = {kGK1, kGK2, kGQ1, kGQ2};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        uint64_t x[P];
        load_pairs<P>(vec + which[j] * L::kD, rg, x);
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[j][c] = mul2(S[0][c], x[0]);
#pragma unroll
        for (int p = 1; p < P; ++p)
#pragma unroll
          for (int c = 0; c < 4; ++c) acc[j][c] = fma2(S[p][c], x[p], acc[j][c]);
      }
      // decay the state while the sums travel
      {
        uint64_t gg[P];
        load_pairs<P>(vec + kGG * L::kD, rg, gg);
#pragma unroll
        for (int p = 0; p < P; ++p)
#pragma unroll
          for (int c = 0; c < 4; ++c) S[p][c] = mul2(S[p][c], gg[p]);
      }
      float x8[8], x4[4], x2[2], x;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const float sk1 = half_sum(acc[0][c]), sk2 = half_sum(acc[1][c]), sq1 = half_sum(acc[2][c]), sq2 = half_sum(acc[3][c]);
        x8[c] = (is_q ? sq1 : sk1) + __shfl_xor_sync(0xffffffffu, is_q ? sk1 : sq1, 8);
        x8[4 + c] = (is_q ? sq2 : sk2) + __shfl_xor_sync(0xffffffffu, is_q ? sk2 : sq2, 8);
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) x4[c] = (second ? x8[4 + c] : x8[c]) + __shfl_xor_sync(0xffffffffu, second ? x8[c] : x8[4 + c], 4);
#pragma unroll
      for (int c = 0; c < 2; ++c) x2[c] = (b1 ? x4[2 + c] : x4[c]) + __shfl_xor_sync(0xffffffffu, b1 ? x4[c] : x4[2 + c], 2);
      x = (b0 ? x2[1] : x2[0]) + __shfl_xor_sync(0xffffffffu, b0 ? x2[0] : x2[1], 1);
      const float u1_own = sc.x * (v1 - x);                                           // right in lanes 0-3 of a half
      const float u1s = __shfl_sync(0xffffffffu, u1_own, half + mine);
      const float u2_own = sc.z * (v2 - fmaf(u1s, cross.x, x));                       // right in lanes 4-7
      float u1[4], u2[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) u1[c] = __shfl_sync(0xffffffffu, u1_own, half + c);
#pragma unroll
      for (int c = 0; c < 4; ++c) u2[c] = __shfl_sync(0xffffffffu, u2_own, half + 4 + c);
      {
        uint64_t w1[P], w2[P];
        load_pairs<P>(vec + kW1 * L::kD, rg, w1);
        load_pairs<P>(vec + kW2 * L::kD, rg, w2);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const uint64_t ua = pack2(u1[c], u1[c]), ub = pack2(u2[c], u2[c]);
#pragma unroll
          for (int p = 0; p < P; ++p) S[p][c] = fma2(w2[p], ub, fma2(w1[p], ua, S[p][c]));
        }
      }
      const float u2s = b1 ? (b0 ? u2[3] : u2[2]) : (b0 ? u2[1] : u2[0]);
      const float o = second ? fmaf(u2s, sc.w, fmaf(u1s, cross.y, x)) : fmaf(u1s, sc.y, x);
      const int row = 2 * (i * kTile + t);
      if (writes && row + (second ? 1 : 0) < n) o_dst[static_cast<int64_t>(row) * o_ld] = o;
    }
    if (__syncthreads_or(failed)) break;      // also releases the stage
  }
  if (failed) {
    // let copies in flight land before the CTA's shared memory is released
    for (int s = 0; s < kStages; ++s) ptx::mbar_wait(bars + 8 * s, 0, 20000000ull) || ptx::mbar_wait(bars + 8 * s, 1, 20000000ull);
    return;
  }
  store_state<P, 4>(state, d, e, col, rg, S);
}

// out = rms_norm(o) * w * gate for the rows of sequences >= first: one warp per (row, head).
template <typename T, int VEC, int NJ>
__global__ void __launch_bounds__(256) delta_out_kernel(const B2DeltaArgs a, const B2SeqRows sq, int first) {
  ptx::grid_dep_sync();
  const int64_t idx = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, e = a.vdim;
  const int row = static_cast<int>(idx / a.heads), h = static_cast<int>(idx % a.heads);
  if (row >= sq.rows || sq.row_seq[row] < first) return;
  const float* o = a.o_raw + (static_cast<int64_t>(row) * a.heads + h) * e;
  const T* gate = gate_row<T>(a, row, h);
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
  const float r = rsqrtf(ss / static_cast<float>(e) + a.eps);
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = (lane + 32 * j) * VEC;
    if (c >= e) continue;
    float z[VEC], w[VEC];
    load_f32<VEC>(gate + c, z);
    load_f32<VEC>(a.norm_w + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[j][i] = v[j][i] * r * w[i] * gate_value(a, z[i]);
    store_f32<VEC>(out + c, v[j]);
  }
}

template <int P>
int launch_scan(const B2DeltaArgs& a, const B2SeqRows& s, int first, int n, Status* status, cudaStream_t stream) {
  using L = ScanLayout<P>;
  static DeviceOnce attr_once;
  if (const int rc = attr_once.max_smem(delta_scan_kernel<P>, L::kBytes)) return rc;
  launch_pdl(delta_scan_kernel<P>, dim3((a.vdim + kCols - 1) / kCols, a.heads, n), dim3(128), L::kBytes, stream, a, s, prepared_of(a, s), first, status);
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
  const bool v4 = a.vdim % 4 == 0 && vec4_rows<T>(a.gate, a.ld_gate) && a.ld_out % 4 == 0;
  if (v4 && a.vdim <= 128) launch_pdl(delta_out_kernel<T, 4, 1>, grid, dim3(256), 0, stream, a, s, first);
  else if (v4) launch_pdl(delta_out_kernel<T, 4, 2>, grid, dim3(256), 0, stream, a, s, first);
  else launch_pdl(delta_out_kernel<T, 1, 8>, grid, dim3(256), 0, stream, a, s, first);
  return last_launch_rc();
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int64_t b2_delta_scratch_floats(int heads, int dim, int vdim, int rows, int seqs) {
  return scratch_floats(heads, dim, vdim, rows, seqs);
}

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
