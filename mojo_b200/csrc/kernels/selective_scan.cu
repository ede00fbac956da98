// Selective scan: every channel has a row of states that decay by rates of their own, scaled by the token's step size, and a
// token writes to and reads from all states of all channels through two vectors that the channels share. All of it in f32.
// L neighbouring lanes hold the states of one channel, NS each, in registers. A state's next value needs one multiply-add after
// its last one, everything else runs ahead, so the chain over a prompt's rows is short and is not cut; the decays (one
// exponential per state and row) are most of the work.
//   decode  one row per sequence: states stream through registers, several sequences per CTA, rates stay
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
constexpr int kDecodeSeqs = 8;      // sequences of one decode CTA

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
// One row: S <- 2^(dt rate) S + dtu B; returns S . C over this thread's states.
template <bool EXACT, int N>
__device__ __forceinline__ float scan_row(uint64_t (&S)[N / 2], const uint64_t (&rate)[N / 2], float dt, float dtu, const uint64_t (&B)[N / 2],
                                          const uint64_t (&C)[N / 2]) {
  const uint64_t dt2 = pack2(dt, dt), u2 = pack2(dtu, dtu);
  uint64_t y = 0;
#pragma unroll
  for (int i = 0; i < N / 2; ++i) {
    const float2 x = unpack2(mul2(dt2, rate[i]));
    S[i] = fma2(pack2(decay<EXACT>(x.x), decay<EXACT>(x.y)), S[i], mul2(u2, B[i]));
    y = i == 0 ? mul2(S[i], C[i]) : fma2(S[i], C[i], y);
  }
  return half_sum(y);
}

template <typename T, int L, int NS>
__global__ void __launch_bounds__(kThreads) scan_decode_kernel(const B2SelectiveScanArgs a, const B2SeqRows sq, int n_seqs, Status* status) {
  ptx::grid_dep_sync();
  constexpr int CH = kThreads / L, SP = L * NS;
  const int l = threadIdx.x % L, ch = blockIdx.x * CH + threadIdx.x / L;
  const bool in = ch < a.channels;
  uint64_t rate[NS / 2] = {};
  float bias = 0.0f, d = 0.0f;
  if (in) {
    load_packed<NS>(a.rate + static_cast<int64_t>(ch) * SP + l * NS, rate);
    bias = a.dt_bias[ch];
    d = a.d[ch];
  }
  struct Step { uint64_t S[NS / 2], B[NS / 2], C[NS / 2]; float dt, u, z; float* state; int row; };
  const auto request = [&](int seq) {
    Step s{};
    ConvRow cr;
    s.row = seq < n_seqs ? decode_row(sq, seq, cr, status) : -1;
    if (s.row < 0 || !in) return s;
    s.state = a.state + (static_cast<int64_t>(cr.wr >> 1) * a.channels + ch) * SP + l * NS;
    if (cr.rd >= 0) load_packed<NS>(s.state, s.S);
    float b[NS], c[NS], one[1];
    const T *bp = static_cast<const T*>(a.b) + s.row * a.ld_bc + l * NS, *cp = static_cast<const T*>(a.c) + s.row * a.ld_bc + l * NS;
#pragma unroll
    for (int i = 0; i < NS; i += (NS < 4 ? 2 : 4)) {
      constexpr int V = NS < 4 ? 2 : 4;
      load_f32<V>(bp + i, *reinterpret_cast<float(*)[V]>(b + i));
      load_f32<V>(cp + i, *reinterpret_cast<float(*)[V]>(c + i));
    }
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) {
      s.B[i] = pack2(b[2 * i], b[2 * i + 1]);
      s.C[i] = pack2(c[2 * i], c[2 * i + 1]);
    }
    s.dt = a.dt[s.row * a.ld_dt + ch];
    load_f32<1>(static_cast<const T*>(a.u) + s.row * a.ld_u + ch, one);
    s.u = one[0];
    load_f32<1>(static_cast<const T*>(a.z) + s.row * a.ld_z + ch, one);
    s.z = one[0];
    return s;
  };
  const int seq0 = blockIdx.y * kDecodeSeqs, seq1 = min(n_seqs, seq0 + kDecodeSeqs);
  Step next = request(seq0);
  for (int seq = seq0; seq < seq1; ++seq) {
    Step s = next;
    next = request(seq + 1 < seq1 ? seq + 1 : n_seqs);
    if (s.row < 0) continue;      // uniform per CTA
    const float dt = softplus_fast(s.dt + bias);
    float y = scan_row<sizeof(T) == 4, NS>(s.S, rate, dt, dt * s.u, s.B, s.C);
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (!in) continue;
    store_packed<NS>(s.state, s.S);
    if (l == 0) {
      const float out[1] = {fmaf(d, s.u, y) * ptx::silu(s.z)};
      store_f32<1>(static_cast<T*>(a.out) + s.row * a.ld_out + ch, out);
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
  extern __shared__ __align__(16) float bc_sm[];                                             // [2 buffers][B, C][TR][SP]
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
    float *b_sm = bc_sm + buf * 2 * TR * SP, *c_sm = b_sm + TR * SP;
    float du[kPer][4], gate[kPer][4];
#pragma unroll
    for (int k = 0; k < kPer; ++k) {
      int r, c;
      if (!place(k, r, c)) continue;
      float bias[4], d[4];
      load_f32<4>(a.dt_bias + ch0 + c, bias);
      load_f32<4>(a.d + ch0 + c, d);
      float s[8];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float u = u_in[k].get(i), z = z_in[k].get(i);
        s[2 * i] = r < rows ? softplus_fast(dt_in[k][i] + bias[i]) : 0.0f;      // a row that is not there changes nothing
        s[2 * i + 1] = s[2 * i] * u;
        du[k][i] = d[i] * u;
        gate[k][i] = ptx::silu(z);
      }
      float* to = reinterpret_cast<float*>(&step_sm[buf][r][c]);
      store_f32<4>(to, *reinterpret_cast<float(*)[4]>(s));
      store_f32<4>(to + 4, *reinterpret_cast<float(*)[4]>(s + 4));
    }
#pragma unroll
    for (int k = 0; k < kBcPer; ++k) {
      const int i = threadIdx.x + k * kThreads;
      if (kBc % kThreads != 0 && i >= kBc) continue;
      float b[4], c[4];
#pragma unroll
      for (int v = 0; v < 4; ++v) {
        b[v] = b_in[k].get(v);
        c[v] = c_in[k].get(v);
      }
      store_f32<4>(b_sm + 4 * i, b);
      store_f32<4>(c_sm + 4 * i, c);
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
        y[i] = scan_row<sizeof(T) == 4, NS>(S, rate, s.x, s.y, B, C);
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
int launch(const B2SelectiveScanArgs& a, const B2SeqRows& s, int n_decode, int first, int n_prefill, Status* status, cudaStream_t stream) {
  constexpr int CH = kThreads / L, SP = L * NS, kBcBytes = 4 * tile_rows<L>() * SP * 4;
  const int blocks = (a.channels + CH - 1) / CH;
  if (n_decode > 0)
    launch_pdl(scan_decode_kernel<T, L, NS>, dim3(blocks, (n_decode + kDecodeSeqs - 1) / kDecodeSeqs), dim3(kThreads), 0, stream, a, s, n_decode, status);
  if (n_prefill > 0) {
    static DeviceOnce attr_once;
    if (kBcBytes > 24 * 1024)
      if (const int rc = attr_once.max_smem(scan_kernel<T, L, NS>, kBcBytes)) return rc;
    launch_pdl(scan_kernel<T, L, NS>, dim3(blocks, n_prefill), dim3(kThreads), kBcBytes, stream, a, s, first, status);
  }
  return last_launch_rc();
}

template <typename T>
int dispatch(const B2SelectiveScanArgs& a, const B2SeqRows& s, int n_decode, int first, int n_prefill, Status* status, cudaStream_t stream) {
  // few channels in all: more lanes for each
  const bool few = static_cast<int64_t>(a.channels) * (n_decode + n_prefill) * a.states < 4ll * 128 * 1024;
  switch (a.states) {
    case 4: return launch<T, 2, 2>(a, s, n_decode, first, n_prefill, status, stream);
    case 8: return launch<T, 4, 2>(a, s, n_decode, first, n_prefill, status, stream);
    case 16:
      return few ? launch<T, 8, 2>(a, s, n_decode, first, n_prefill, status, stream) : launch<T, 4, 4>(a, s, n_decode, first, n_prefill, status, stream);
    case 32:
      return few ? launch<T, 16, 2>(a, s, n_decode, first, n_prefill, status, stream) : launch<T, 8, 4>(a, s, n_decode, first, n_prefill, status, stream);
    case 64: return launch<T, 16, 4>(a, s, n_decode, first, n_prefill, status, stream);
    case 128: return launch<T, 32, 4>(a, s, n_decode, first, n_prefill, status, stream);
    case 256: return launch<T, 32, 8>(a, s, n_decode, first, n_prefill, status, stream);
    default: return -kBadArgument;
  }
}

}  // namespace
}  // namespace b2

using namespace b2;

extern "C" int b2_selective_scan(const B2SelectiveScanArgs* a, const B2SeqRows* s, int n_decode, int first, int n_prefill, int f32, Status* status,
                                 cudaStream_t stream) {
  if (s->rows <= 0 || n_decode + n_prefill <= 0) return 0;
  const int64_t esz = f32 ? 4 : 2;
  const auto fits = [](const void* p, int64_t ld, int64_t size) { return p != nullptr && ld % 4 == 0 && reinterpret_cast<uintptr_t>(p) % (4 * size) == 0; };
  if (a->channels <= 0 || a->channels % 8 != 0 || n_decode < 0 || n_prefill < 0 || first < n_decode || first + n_prefill > s->seqs || n_decode > 8 * 65535 ||
      n_prefill > 65535 || a->state == nullptr || a->rate == nullptr || a->dt_bias == nullptr || a->d == nullptr || !fits(a->dt, a->ld_dt, 4) ||
      !fits(a->u, a->ld_u, esz) || !fits(a->z, a->ld_z, esz) || !fits(a->b, a->ld_bc, esz) || !fits(a->c, a->ld_bc, esz) || !fits(a->out, a->ld_out, esz))
    return -kBadArgument;
  return f32 ? dispatch<float>(*a, *s, n_decode, first, n_prefill, status, stream)
             : dispatch<__nv_bfloat16>(*a, *s, n_decode, first, n_prefill, status, stream);
}
