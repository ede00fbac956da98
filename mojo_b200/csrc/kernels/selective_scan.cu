// Selective scan: every channel has a row of states that decay by rates of their own, scaled by the token's step size, and a
// token writes to and reads from all states of all channels through two vectors that the channels share. All of it in f32.
// L neighbouring lanes hold the states of one channel, NS each, in registers. A state's next value needs one multiply-add after
// its last one, everything else runs ahead, so the chain over a prompt's rows is short and is not cut; the decays (one
// exponential per state and row) are most of the work.
//   decode  one row per sequence: a CTA keeps its channels' rates and walks over sequences, the next ones' states on their way
//   scan    any number of rows: tiles of rows are brought into shared memory as f32 while the tile before is computed; the L
//           partial sums of L rows are exchanged at once, so that each lane ends up with one row's
#include <cstdint>
#include "b2/elem.cuh"
#include "b2/launch.h"
#include "b2/mixers.h"
#include "b2/ptx.cuh"
#include "b2/recurrence.cuh"
#include "b2/vec.cuh"

namespace b2 {
namespace {

constexpr int kThreads = 128;
constexpr int kAhead = 4;           // sequences on their way to a decode CTA
constexpr int kMaxSeqs = 128;       // sequences of one decode CTA

// N values in pairs. Eight states are one 32-byte access.
template <int N>
__device__ __forceinline__ void load_packed(const __nv_bfloat16* p, uint64_t (&v)[N / 2]) {
  constexpr int V = N < 4 ? 2 : 4;
#pragma unroll
  for (int i = 0; i < N; i += V) {
    float f[V];
    load_f32<V>(p + i, f);
#pragma unroll
    for (int j = 0; j < V / 2; ++j) v[i / 2 + j] = pack2(f[2 * j], f[2 * j + 1]);
  }
}
template <int N>
__device__ __forceinline__ void load_packed(const float* p, uint64_t (&v)[N / 2]) {
  if constexpr (N == 2) {
    v[0] = *reinterpret_cast<const uint64_t*>(p);
  } else {
#pragma unroll
    for (int i = 0; i < N / 4; ++i) {
      const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(p + 4 * i);
      v[2 * i] = t.x;
      v[2 * i + 1] = t.y;
    }
  }
}
template <int N>
__device__ __forceinline__ void store_packed(float* p, const uint64_t (&v)[N / 2]) {
  if constexpr (N == 2) {
    *reinterpret_cast<uint64_t*>(p) = v[0];
  } else {
#pragma unroll
    for (int i = 0; i < N / 4; ++i) {
      ulonglong2 t;
      t.x = v[2 * i];
      t.y = v[2 * i + 1];
      *reinterpret_cast<ulonglong2*>(p + 4 * i) = t;
    }
  }
}
// 2^x for x <= 0. The special-function unit's error has the same sign over wide stretches, which adds up in a state that decays
// slowly: `EXACT` takes the Taylor series of e^t there.
template <bool EXACT>
__device__ __forceinline__ float decay(float x) {
  if constexpr (EXACT) {
    const float t = x * ptx::kLn2;
    if (t > -0.25f) {
      float p = fmaf(t, 1.0f / 720, 1.0f / 120);
      p = fmaf(t, p, 1.0f / 24);
      p = fmaf(t, p, 1.0f / 6);
      p = fmaf(t, p, 0.5f);
      p = fmaf(t, p, 1.0f);
      return fmaf(t, p, 1.0f);
    }
  }
  return ptx::ex2(x);
}
// One row: S <- 2^(dt rate) S + u B, dt and u twice each; returns S . C over this thread's states.
template <bool EXACT, int N>
__device__ __forceinline__ float scan_row(uint64_t (&S)[N / 2], const uint64_t (&rate)[N / 2], uint64_t dt2, uint64_t u2, const uint64_t (&B)[N / 2],
                                          const uint64_t (&C)[N / 2]) {
  uint64_t y = 0;
#pragma unroll
  for (int i = 0; i < N / 2; ++i) {
    const float2 x = unpack2(mul2(dt2, rate[i]));
    S[i] = fma2(pack2(decay<EXACT>(x.x), decay<EXACT>(x.y)), S[i], mul2(u2, B[i]));
    y = i == 0 ? mul2(S[i], C[i]) : fma2(S[i], C[i], y);
  }
  return half_sum(y);
}

// The states of a thread in global memory: 32 bytes at once where there are so many.
template <int N>
__device__ __forceinline__ void load_states(const float* p, uint64_t (&v)[N / 2]) {
  if constexpr (N == 8) asm volatile("ld.global.v4.b64 {%0, %1, %2, %3}, [%4];" : "=l"(v[0]), "=l"(v[1]), "=l"(v[2]), "=l"(v[3]) : "l"(p));
  else load_packed<N>(p, v);
}
template <int N>
__device__ __forceinline__ void store_states(float* p, const uint64_t (&v)[N / 2]) {
  if constexpr (N == 8) asm volatile("st.global.v4.b64 [%0], {%1, %2, %3, %4};" ::"l"(p), "l"(v[0]), "l"(v[1]), "l"(v[2]), "l"(v[3]) : "memory");
  else store_packed<N>(p, v);
}

template <typename T, int L, int NS>
__global__ void __launch_bounds__(kThreads) scan_decode_kernel(const B2SelectiveScanArgs a, const B2SeqRows sq, int n_seqs, int per_cta, Status* status) {
  ptx::grid_dep_sync();
  constexpr int CH = kThreads / L, SP = L * NS, V = NS < 4 ? 2 : 4;
  const int l = threadIdx.x % L, ch = blockIdx.x * CH + threadIdx.x / L;
  const bool in = ch < a.channels;
  // the places of this CTA's sequences: row (-1: none), state slot, whether it starts from zero
  __shared__ int row_sm[kMaxSeqs], slot_sm[kMaxSeqs];
  const int seq0 = blockIdx.y * per_cta, n = min(per_cta, n_seqs - seq0);
  if (static_cast<int>(threadIdx.x) < n) {
    ConvRow cr;
    const int row = decode_row(sq, seq0 + threadIdx.x, cr, status);
    row_sm[threadIdx.x] = row;
    slot_sm[threadIdx.x] = row < 0 ? 0 : (cr.wr >> 1) * 2 + (cr.rd < 0 ? 1 : 0);
  }
  __syncthreads();
  uint64_t S[kAhead][NS / 2];
  RawVec<T, V> B[kAhead][NS / V], C[kAhead][NS / V];
  float dt[kAhead];
  RawVec<T, 2> uz[kAhead];      // two values in one register
  const auto state_of = [&](int q) { return a.state + (static_cast<int64_t>(slot_sm[q] >> 1) * a.channels + ch) * SP + l * NS; };
  const auto request = [&](int q, int at) {
    const int row = q < n ? row_sm[q] : -1;
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) S[at][i] = 0;
    if (row < 0 || !in) return;
    if (!(slot_sm[q] & 1)) load_states<NS>(state_of(q), S[at]);
    const T *bp = static_cast<const T*>(a.b) + row * a.ld_bc + l * NS, *cp = static_cast<const T*>(a.c) + row * a.ld_bc + l * NS;
#pragma unroll
    for (int i = 0; i < NS / V; ++i) {
      B[at][i].load(bp + i * V);
      C[at][i].load(cp + i * V);
    }
    dt[at] = a.dt[row * a.ld_dt + ch];
    uz[at].set(static_cast<const T*>(a.u)[row * a.ld_u + ch], static_cast<const T*>(a.z)[row * a.ld_z + ch]);
  };
#pragma unroll
  for (int q = 0; q < kAhead; ++q) request(q, q);
  uint64_t rate[NS / 2] = {};
  float bias = 0.0f, d = 0.0f;
  if (in) {
    load_states<NS>(a.rate + static_cast<int64_t>(ch) * SP + l * NS, rate);
    bias = a.dt_bias[ch];
    d = a.d[ch];
  }
  for (int q0 = 0; q0 < n; q0 += kAhead) {
#pragma unroll
    for (int at = 0; at < kAhead; ++at) {
      const int q = q0 + at, row = q < n ? row_sm[q] : -1;      // uniform per CTA
      if (row >= 0) {
        float y = 0.0f, u = 0.0f, z = 0.0f;
        if (in) {
          uint64_t b[NS / 2], c[NS / 2];
#pragma unroll
          for (int i = 0; i < NS / 2; ++i) {
            b[i] = pack2(B[at][2 * i / V].get(2 * i % V), B[at][2 * i / V].get(2 * i % V + 1));
            c[i] = pack2(C[at][2 * i / V].get(2 * i % V), C[at][2 * i / V].get(2 * i % V + 1));
          }
          u = uz[at].get(0);
          z = uz[at].get(1);
          const float step = softplus_fast(dt[at] + bias);
          y = scan_row<sizeof(T) == 4, NS>(S[at], rate, pack2(step, step), pack2(step * u, step * u), b, c);
          store_states<NS>(state_of(q), S[at]);
        }
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        if (in && l == 0) {
          const float out[1] = {fmaf(d, u, y) * ptx::silu(z)};
          store_f32<1>(static_cast<T*>(a.out) + row * a.ld_out + ch, out);
        }
      }
      request(q + kAhead, at);
    }
  }
}

template <int L>
constexpr int tile_rows() { return L == 8 || L == 32 ? 32 : 16; }

template <typename T, int L, int NS>
__global__ void __launch_bounds__(kThreads) scan_kernel(const B2SelectiveScanArgs a, const B2SeqRows sq, int first, Status* status) {
  ptx::grid_dep_sync();
  constexpr int CH = kThreads / L, SP = L * NS, TR = tile_rows<L>();
  constexpr int kVecs = TR * CH / 4, kPer = (kVecs + kThreads - 1) / kThreads;               // quadruples of channels in a tile
  constexpr int kBc = TR * SP / 4, kBcPer = (kBc + kThreads - 1) / kThreads;                 // of states, B and C alike
  __shared__ __align__(16) float2 step_sm[2][TR][CH];                                        // dt, dt u
  __shared__ __align__(16) float y_sm[TR][CH];
  extern __shared__ __align__(16) uint8_t bc_raw[];                                          // [2 buffers][B, C][TR][SP]
  T* bc_sm = reinterpret_cast<T*>(bc_raw);
  const int seq = first + blockIdx.y, ch0 = blockIdx.x * CH;
  const int l = threadIdx.x % L, cl = threadIdx.x / L, ch = ch0 + cl;
  const int begin = sq.seq_rows[2 * seq];
  ConvRow cr;
  if (sq.seq_rows[2 * seq + 1] <= begin || !cr.load(sq, seq, begin, sq.banks, status)) return;      // uniform per CTA
  const int n = cr.end - cr.begin, n_tiles = (n + TR - 1) / TR;
  const bool in = ch < a.channels;
  uint64_t rate[NS / 2] = {}, S[NS / 2] = {};
  float* state = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.channels + (in ? ch : 0)) * SP + l * NS;
  if (in) {
    load_packed<NS>(a.rate + static_cast<int64_t>(ch) * SP + l * NS, rate);
    if (cr.rd >= 0) load_packed<NS>(state, S);
  }
  // this thread's share of a tile: rows and channel quadruples, for staging as well as for the results
  const auto place = [&](int k, int& r, int& c) {
    const int i = threadIdx.x + k * kThreads;
    r = i / (CH / 4);
    c = i % (CH / 4) * 4;
    return (kVecs % kThreads == 0 || i < kVecs) && ch0 + c < a.channels;
  };
  float dt_in[kPer][4];
  RawVec<T, 4> u_in[kPer], z_in[kPer], b_in[kBcPer], c_in[kBcPer];
  const auto request = [&](int tile) {
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
      int r, c;
      const bool ok = place(k, r, c) && tile * TR + r < n;
#pragma unroll
      for (int i = 0; i < 4; ++i) dt_in[k][i] = 0.0f;
      u_in[k].zero();
      z_in[k].zero();
      if (!ok) continue;
      const int64_t row = begin + tile * TR + r;
      load_f32<4>(a.dt + row * a.ld_dt + ch0 + c, dt_in[k]);
      u_in[k].load(static_cast<const T*>(a.u) + row * a.ld_u + ch0 + c);
      z_in[k].load(static_cast<const T*>(a.z) + row * a.ld_z + ch0 + c);
    }
#pragma unroll
    for (int k = 0; k < kBcPer; ++k) {
      const int i = threadIdx.x + k * kThreads, r = i / (SP / 4), c = i % (SP / 4) * 4;
      b_in[k].zero();
      c_in[k].zero();
      if (i >= kBc || tile * TR + r >= n) continue;
      const int64_t row = begin + tile * TR + r;
      b_in[k].load(static_cast<const T*>(a.b) + row * a.ld_bc + c);
      c_in[k].load(static_cast<const T*>(a.c) + row * a.ld_bc + c);
    }
  };
  request(0);
  for (int tile = 0; tile < n_tiles; ++tile) {
    const int buf = tile & 1, rows = min(TR, n - tile * TR);
    T *b_sm = bc_sm + buf * 2 * TR * SP, *c_sm = b_sm + TR * SP;
    float du[kPer][4], gate[kPer][4];
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
      int r, c;
      if (!place(k, r, c)) continue;
      float bias[4], d[4];
      load_f32<4>(a.dt_bias + ch0 + c, bias);
      load_f32<4>(a.d + ch0 + c, d);
      float2 step[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float u = u_in[k].get(i), z = z_in[k].get(i);
        const float dt = r < rows ? softplus_fast(dt_in[k][i] + bias[i]) : 0.0f;      // a row that is not there changes nothing
        step[i] = make_float2(dt, dt * u);
        du[k][i] = d[i] * u;
        gate[k][i] = ptx::silu(z);
      }
      *reinterpret_cast<float4*>(&step_sm[buf][r][c]) = make_float4(step[0].x, step[0].y, step[1].x, step[1].y);
      *reinterpret_cast<float4*>(&step_sm[buf][r][c + 2]) = make_float4(step[2].x, step[2].y, step[3].x, step[3].y);
    }
#pragma unroll
    for (int k = 0; k < kBcPer; ++k) {
      const int i = threadIdx.x + k * kThreads;
      if (kBc % kThreads != 0 && i >= kBc) continue;
      b_in[k].store(b_sm + 4 * i);
      c_in[k].store(c_sm + 4 * i);
    }
    if (tile + 1 < n_tiles) request(tile + 1);
    __syncthreads();      // also: the results of the tile before have been read
    for (int r0 = 0; r0 < rows; r0 += L) {
      float y[L];
#pragma unroll
      for (int i = 0; i < L; ++i) {
        const float2 s = step_sm[buf][r0 + i][cl];
        uint64_t B[NS / 2], C[NS / 2];
        load_packed<NS>(b_sm + (r0 + i) * SP + l * NS, B);
        load_packed<NS>(c_sm + (r0 + i) * SP + l * NS, C);
        y[i] = scan_row<sizeof(T) == 4, NS>(S, rate, pack2(s.x, s.x), pack2(s.y, s.y), B, C);
      }
      // the sums over the lanes of a channel: a lane keeps the half of the rows that its bit names
#pragma unroll
      for (int w = L / 2; w > 0; w >>= 1) {
        const bool hi = l & w;
#pragma unroll
        for (int i = 0; i < w; ++i) y[i] = (hi ? y[i + w] : y[i]) + __shfl_xor_sync(0xffffffffu, hi ? y[i] : y[i + w], w);
      }
      y_sm[r0 + l][cl] = y[0];
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
      int r, c;
      if (!place(k, r, c) || r >= rows) continue;
      float y[4];
      load_f32<4>(&y_sm[r][c], y);
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] = (y[i] + du[k][i]) * gate[k][i];
      store_f32<4>(static_cast<T*>(a.out) + static_cast<int64_t>(begin + tile * TR + r) * a.ld_out + ch0 + c, y);
    }
  }
  if (in) store_packed<NS>(state, S);
}

template <typename T, int L, int NS>
int launch_decode(const B2SelectiveScanArgs& a, const B2SeqRows& s, int n, Status* status, cudaStream_t stream) {
  constexpr int CH = kThreads / L;
  const int64_t blocks = (a.channels + CH - 1) / CH;
  const int64_t runs = blocks < 4 * kNumSMs ? 4 * kNumSMs / blocks : 1;      // of sequences, so that all CTAs fit at once
  int64_t per = (n + runs - 1) / runs;
  if (per > kMaxSeqs) per = kMaxSeqs;
  launch_pdl(scan_decode_kernel<T, L, NS>, dim3(static_cast<unsigned>(blocks), static_cast<unsigned>((n + per - 1) / per)), dim3(kThreads), 0, stream, a, s, n,
             static_cast<int>(per), status);
  return last_launch_rc();
}
template <typename T>
int dispatch_decode(const B2SelectiveScanArgs& a, const B2SeqRows& s, int n, Status* status, cudaStream_t stream) {
  switch (a.states) {
    case 4: return launch_decode<T, 1, 4>(a, s, n, status, stream);
    case 8: return launch_decode<T, 1, 8>(a, s, n, status, stream);
    case 16: return launch_decode<T, 2, 8>(a, s, n, status, stream);
    case 32: return launch_decode<T, 4, 8>(a, s, n, status, stream);
    case 64: return launch_decode<T, 8, 8>(a, s, n, status, stream);
    case 128: return launch_decode<T, 16, 8>(a, s, n, status, stream);
    case 256: return launch_decode<T, 32, 8>(a, s, n, status, stream);
    default: return -kBadArgument;
  }
}

template <typename T, int L, int NS>
int launch_scan(const B2SelectiveScanArgs& a, const B2SeqRows& s, int first, int n, Status* status, cudaStream_t stream) {
  constexpr int CH = kThreads / L, kBcBytes = 4 * tile_rows<L>() * L * NS * static_cast<int>(sizeof(T));
  static DeviceOnce attr_once;
  if (kBcBytes > 24 * 1024)
    if (const int rc = attr_once.max_smem(scan_kernel<T, L, NS>, kBcBytes)) return rc;
  launch_pdl(scan_kernel<T, L, NS>, dim3((a.channels + CH - 1) / CH, n), dim3(kThreads), kBcBytes, stream, a, s, first, status);
  return last_launch_rc();
}
template <typename T>
int dispatch_scan(const B2SelectiveScanArgs& a, const B2SeqRows& s, int first, int n, Status* status, cudaStream_t stream) {
  // few channels in all: more lanes for each
  const bool few = static_cast<int64_t>(a.channels) * n * a.states < 4ll * 128 * 1024;
  switch (a.states) {
    case 4: return launch_scan<T, 2, 2>(a, s, first, n, status, stream);
    case 8: return launch_scan<T, 4, 2>(a, s, first, n, status, stream);
    case 16: return few ? launch_scan<T, 8, 2>(a, s, first, n, status, stream) : launch_scan<T, 4, 4>(a, s, first, n, status, stream);
    case 32: return few ? launch_scan<T, 16, 2>(a, s, first, n, status, stream) : launch_scan<T, 8, 4>(a, s, first, n, status, stream);
    case 64: return launch_scan<T, 16, 4>(a, s, first, n, status, stream);
    case 128: return launch_scan<T, 32, 4>(a, s, first, n, status, stream);
    case 256: return launch_scan<T, 32, 8>(a, s, first, n, status, stream);
    default: return -kBadArgument;
  }
}

template <typename T>
int dispatch(const B2SelectiveScanArgs& a, const B2SeqRows& s, int n_decode, int first, int n_prefill, Status* status, cudaStream_t stream) {
  if (n_decode > 0)
    if (const int rc = dispatch_decode<T>(a, s, n_decode, status, stream)) return rc;
  return n_prefill > 0 ? dispatch_scan<T>(a, s, first, n_prefill, status, stream) : 0;
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_selective_scan(const B2SelectiveScanArgs* a, const B2SeqRows* s, int n_decode, int first, int n_prefill, int f32, Status* status,
                                 cudaStream_t stream) {
  if (s->rows <= 0 || n_decode + n_prefill <= 0) return 0;
  const int64_t esz = f32 ? 4 : 2;
  const auto fits = [](const void* p, int64_t ld, int64_t size) { return p != nullptr && ld % 4 == 0 && reinterpret_cast<uintptr_t>(p) % (4 * size) == 0; };
  if (a->channels <= 0 || a->channels % 8 != 0 || n_decode < 0 || n_prefill < 0 || first < n_decode || first + n_prefill > s->seqs || n_decode > 65535 ||
      n_prefill > 65535 || a->state == nullptr || a->rate == nullptr || a->dt_bias == nullptr || a->d == nullptr || !fits(a->dt, a->ld_dt, 4) ||
      !fits(a->u, a->ld_u, esz) || !fits(a->z, a->ld_z, esz) || !fits(a->b, a->ld_bc, esz) || !fits(a->c, a->ld_bc, esz) || !fits(a->out, a->ld_out, esz))
    return -kBadArgument;
  return f32 ? dispatch<float>(*a, *s, n_decode, first, n_prefill, status, stream)
             : dispatch<__nv_bfloat16>(*a, *s, n_decode, first, n_prefill, status, stream);
}
