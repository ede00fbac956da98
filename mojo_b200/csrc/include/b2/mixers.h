// C launch API of the sequence-mixing kernels beyond plain attention: residual streams with learned mixing
// (hyper-connections), or normalised after the sum, short causal convolutions or norms in front of attention, the gated delta rule,
// gated linear attention, the selective scan, and the 32-bit forms of the matrix product and of paged attention. Conventions as in b2/api.h: raw device pointers, a stream, 0 or
// a negative code back. `f32` selects the element type of activations and caches (0: bf16, 1: f32); parameters that
// enter 32-bit arithmetic (norm weights, mixing coefficients, convolution taps, decay constants) are always f32.
#pragma once
#include <cstdint>
#include <cuda_runtime.h>
#include "b2/api.h"
#include "b2/status.h"

#ifdef __cplusplus
extern "C" {
#endif

// Where the sequences of a step lie in its flat token rows, and which recurrent-state banks they use.
//   row_seq   [rows]     sequence of each row, -1 for padding
//   seq_rows  [seqs, 2]  first row and one past the last row (equal: unused entry)
//   seq_state [seqs, 2]  bank to read (-1: no history) and bank to write (-1: unused entry); bank = 2 * slot + parity
struct B2SeqRows {
  const int32_t* row_seq;
  const int32_t* seq_rows;
  const int32_t* seq_state;
  int32_t rows, seqs, banks;
};

// Residual streams x [rows, streams, width] f32. For every row: x_t <- sum_s mix[s, t] x_s + out[t] y (skipped when y is
// null), then h = rms_norm(sum_s in[s] x_s) * weight. With `ids` the streams start as embed[id] * embed_scale instead of
// being read. `store` writes the new streams back. With `rows_index` only those rows are processed and h is compact.
// Columns from `mean_width` up to `width` are zero padding that the mean leaves out.
struct B2HyperArgs {
  float* x;
  const void* y;
  const float* mix;
  const float* out;
  const float* in;
  const float* weight;
  void* h;
  const int64_t* ids;
  const void* embed;
  const int64_t* rows_index;
  float embed_scale, eps;
  int32_t n_out, rows, width, mean_width, streams, vocab, store;
};
int b2_hyper_norm(const B2HyperArgs* a, int f32, b2::Status* status, cudaStream_t stream);

// One f32 residual stream x [rows, width] with a scale per channel. For every row: x += y_scale * (y + sum_j w[j] e[slot[j]]),
// where y (a sublayer's output) and the expert rows e (`top` of them per row, w and slot [rows, top]) may each be null;
// a row of e with slot -1 is own[row]. `gated` (may be null) is one more addend with a factor sigmoid(gate[row * ld_gate]); y_scale
// null: one. Then h = rms_norm(x) * weight, layer_norm(x) * weight + bias where a bias is given, or x itself rounded where weight
// is null. With `ids` x starts as
// embed[id] * embed_scale (+ bigram[(prev * mul_prev + id * mul_cur) mod buckets], or its last row, number `buckets`, where
// prev is -1) instead of being read, and x0 (may be null) receives a rounded copy of that. `store` writes x back. With
// `rows_index` only those rows are processed and h is compact. Columns from `mean_width` up to `width` are zero padding.
struct B2ResidualArgs {
  float* x;
  const void* y;
  const void* experts;
  const int32_t* expert_slot;
  const float* expert_w;
  const float* y_scale;
  const float* weight;
  void* h;
  const int64_t* ids;
  const void* embed;
  const int32_t* prev;
  const void* bigram;
  void* x0;
  const int64_t* rows_index;
  const float* bias;
  const void* own;
  const void* gated;
  const float* gate;
  int64_t ld_h, ld_x0, mul_prev, mul_cur, buckets, ld_gate;
  float embed_scale, eps;
  int32_t top, expert_rows, n_out, rows, width, mean_width, vocab, store;
};
int b2_residual_norm(const B2ResidualArgs* a, int f32, b2::Status* status, cudaStream_t stream);

// One f32 residual stream that is normalised after the sum. For every row and each of `groups` equal runs of its mean_width columns:
//   v = alpha x + y_scale * (y + sum_j w[j] e[slot[j]])        (y, experts, w and y_scale may each be null: nothing, 1)
//   x_out = v / sqrt(mean(v^2) + eps) * weight                 (weight null: v)
//   h = x_out + conv(x_out)                                    (conv_w null: x_out)
// With `ids` v = embed[id] + pos_table[position] instead. `then` is the weight of one more such norm, ahead of the convolution. The
// convolution is causal over a sequence's rows, per column: conv_w f32 [taps, width], at most 16 taps; conv_state f32 [banks, taps - 1,
// width]. x and x_out are different buffers [rows, width]. With `rows_index` only those rows, h compact, no convolution and no x_out;
// otherwise rows of no sequence read as zero. Columns from mean_width on are left alone.
struct B2PostNormArgs {
  const float* x;
  float* x_out;
  const void* y;
  const void* experts;
  const int32_t* expert_slot;   // [rows, top]
  const float* expert_w;        // [rows, top]
  const float* y_scale;
  const float* weight;
  const float* then;
  const float* conv_w;
  float* conv_state;
  void* h;
  const int64_t* ids;
  const void* embed;
  const void* pos_table;        // [max_pos, width]
  const int32_t* positions;
  const int64_t* rows_index;
  float alpha, eps;
  int32_t top, expert_rows, n_out, rows, width, mean_width, groups, vocab, max_pos, taps;
};
int b2_post_norm(const B2PostNormArgs* a, const B2SeqRows* s, int f32, b2::Status* status, cudaStream_t stream);

// Short causal convolution on the q | k | v channels of a projection, rotary embedding on q and k, RMS norm of each q and k
// head (no weight), and the scatter of k and v into the paged cache; one launch. proj [rows, ld]: the channels start at
// column 0 in the order q (heads * dim), k (kv_heads * dim), v (kv_heads * vdim); kv_heads == 0: queries only.
// conv_w f32 [taps, channels]; conv_state [banks, taps - 1, channels] (null when taps == 1).
// q_out [rows, heads * pad_dim], caches [pages, kv_heads, page_size, pad_dim / pad_vdim]; columns past dim are zero.
struct B2ConvQkvArgs {
  const void* proj;
  int64_t ld;
  const float* conv_w;
  void* conv_state;
  const float* cos_sin;       // [max_pos, rot]
  const int32_t* positions;   // [rows]
  const int64_t* slots;       // [rows], -1: nothing is cached
  void* q_out;
  void* k_cache;
  void* v_cache;
  int64_t num_slots;
  int32_t heads, kv_heads, dim, vdim, pad_dim, pad_vdim, rot, taps, page_size, max_pos;
  float eps;
};
int b2_conv_qkv(const B2ConvQkvArgs* a, const B2SeqRows* s, int f32, b2::Status* status, cudaStream_t stream);

// Front end of attention with norms over whole rows: biases on the q | k | v columns of a projection, one RMS norm (weights
// q_norm, k_norm) over all q columns of a row and one over its k columns, rotary embedding of the first `rot` columns of every q
// and k head (halves pair up), scatter of k and v into the paged cache. Layouts as above; bias f32 [channels].
struct B2NormQkvArgs {
  const void* proj;
  int64_t ld;
  const float* bias;
  const float* q_norm;
  const float* k_norm;
  const float* cos_sin;       // [max_pos, rot]
  const int32_t* positions;   // [rows]
  const int64_t* slots;       // [rows], -1: nothing is cached
  void* q_out;
  void* k_cache;
  void* v_cache;
  int64_t num_slots;
  int32_t rows, heads, kv_heads, dim, vdim, pad_dim, pad_vdim, rot, page_size, max_pos;
  float eps;
};
int b2_norm_qkv(const B2NormQkvArgs* a, int f32, b2::Status* status, cudaStream_t stream);

// Front end of attention with norms per head: RMS norm of every q and k head (weights q_norm, k_norm [dim] for all of them), scatter of
// k and of the values into the paged cache. proj [rows, ld]: q (heads * dim) | k (kv_heads * dim) from column 0, values (kv_heads *
// vdim) from column v_off, which may be the keys' own: then the values are the keys as projected. Layouts as above.
struct B2HeadNormArgs {
  const void* proj;
  int64_t ld;
  const float* q_norm;
  const float* k_norm;
  const int64_t* slots;       // [rows], -1: nothing is cached
  void* q_out;
  void* k_cache;
  void* v_cache;
  int64_t num_slots;
  int32_t rows, heads, kv_heads, dim, vdim, v_off, pad_dim, pad_vdim, page_size;
  float eps;
};
int b2_head_norm_qkv(const B2HeadNormArgs* a, int f32, b2::Status* status, cudaStream_t stream);

// out[t, c] = silu(conv(proj)[t, c] + bias[c]) for `channels` columns of proj, a causal convolution over a sequence's rows;
// conv_w f32 [taps, channels], conv_state [banks, taps - 1, channels] like proj.
struct B2ConvSiluArgs {
  const void* proj;
  int64_t ld;
  const float* conv_w;
  const float* bias;          // may be null
  void* conv_state;
  void* out;
  int64_t ld_out;
  int32_t channels, taps;
};
int b2_conv_silu(const B2ConvSiluArgs* a, const B2SeqRows* s, int f32, b2::Status* status, cudaStream_t stream);

// Selective scan. Per channel c with `states` states, all of it in f32:
//   dt = softplus(dt_logit + dt_bias),  S[n] <- 2^(dt rate[c, n]) S[n] + dt u B[n],  y = sum_n S[n] C[n] + D u,  out = y silu(z)
// rate f32 [channels, states] = -exp(A_log) log2(e). dt f32 [rows, ld_dt]; u, z, out [rows, channels] and B, C [rows, states] with row
// strides. channels % 8 == 0, states one of 4, 8, 16, ... 256 (padding: rate, B and C zero), every row 16-byte aligned (8 for bf16).
// state f32 [slots, channels, states], updated in place. Sequences as for the delta rule below.
struct B2SelectiveScanArgs {
  const float* dt;
  const void* u;
  const void* z;
  const void* b;
  const void* c;
  int64_t ld_dt, ld_u, ld_z, ld_bc, ld_out;
  const float* rate;
  const float* dt_bias;
  const float* d;
  float* state;
  void* out;
  int32_t channels, states;
};
int b2_selective_scan(const B2SelectiveScanArgs* a, const B2SeqRows* s, int n_decode, int first, int n_prefill, int f32, b2::Status* status,
                      cudaStream_t stream);

// Gated linear attention. Per head, with S [dim, vdim], all of it in f32:
//   a = sigmoid(z + decay_bias)^(1 / tau) (one per key channel),  S <- diag(a) S + k v^T,  o = S^T q dim^-0.5
// out = rms_norm(o) * norm_w * silu(gate) * out_scale. proj [rows, ld]: q | k (heads * dim each) | v | gate (heads * vdim each)
// from column 0; z f32 [rows, ld_z]; state f32 [slots, heads, dim, vdim], updated in place.
struct B2GatedLinearArgs {
  const void* proj;
  const float* z;
  int64_t ld, ld_z;
  const float* decay_bias;    // [heads * dim]
  const float* norm_w;        // [vdim]
  float* state;
  float* scratch;             // b2_gated_linear_scratch_floats floats (prompt chunks only)
  void* out;                  // [rows, ld_out], heads * vdim columns
  int64_t ld_out;
  int32_t heads, dim, vdim;
  float inv_tau, eps, out_scale;
};
int64_t b2_gated_linear_scratch_floats(int heads, int dim, int vdim, int rows, int all_seqs, int seqs);      // seqs: those with chunks
int b2_gated_linear_prefill_launches(int heads, int vdim, int rows, int seqs);
// Sequences as for the delta rule below: [0, n_decode) have one row each, [first, first + n_prefill) any number.
int b2_gated_linear(const B2GatedLinearArgs* a, const B2SeqRows* s, int n_decode, int first, int n_prefill, int f32, b2::Status* status,
                    cudaStream_t stream);

// Gated delta rule with one decay per key channel, or one per head. Per head, with S [dim, vdim]:
//   S <- g * S (rows), u = beta (v - S^T k), S <- S + k u^T, o = S^T q
// proj [rows, ld]: q (kv_heads * dim) | k | v (heads * vdim) from column 0, the step-size logits at column b_off;
// decay [rows, ld_decay]: decay inputs (heads * dim; head_decay: heads); gate [rows, ld_gate]: output-gate logits (heads * vdim).
// q, k, v pass the short convolution and silu; q, k become unit vectors, q times dim^-0.5; beta = sigmoid(b);
// g = exp(neg_rate[h] * softplus(decay input + dt_bias)). out = rms_norm(o) * norm_w * f(gate), f the sigmoid or (gate_silu) silu.
// state f32 [slots, heads, dim, vdim], updated in place; conv_state as above.
struct B2DeltaArgs {
  const void* proj;
  const void* decay;
  const void* gate;
  int64_t ld, ld_decay, ld_gate;
  const float* conv_w;
  void* conv_state;
  const float* neg_rate;      // [heads] = -exp(A_log)
  const float* dt_bias;       // [heads * dim], head_decay: [heads]
  const float* norm_w;        // [vdim]
  float* state;
  float* scratch;             // b2_delta_scratch_floats floats: prepared rows
  float* o_raw;               // [rows, heads * vdim], outputs of the scan before norm and gate
  void* out;                  // [rows, ld_out], heads * vdim columns
  int64_t ld_out;
  int32_t b_off, heads, kv_heads, dim, vdim, taps, head_decay, gate_silu;
  float eps;
};
int64_t b2_delta_scratch_floats(int heads, int dim, int vdim, int rows, int seqs);
// Sequences [0, n_decode) of the step have one row each (state read and written once, output finished in the same kernel);
// sequences [first, first + n_prefill) any number of rows (scan, then output norm and gate). The rows of all sequences are
// prepared by one launch ahead of both.
int b2_delta_rule(const B2DeltaArgs* a, const B2SeqRows* s, int n_decode, int first, int n_prefill, int f32, b2::Status* status,
                  cudaStream_t stream);

// Y[M, N] = X[M, K] W[N, K]^T in true f32 (FMA, no reduced-precision matrix mode), `batch` such products side by side: product
// b reads x columns b * K ..., weight rows b * N ... and writes y columns b * N .... Epilogue NONE, RELU2 or SOFTCAP
// (B2Epilogue); then y is multiplied by sigmoid(gate) element by element where a gate [M, batch * N] is given, or product by
// product (`gate_heads`, gate [M, batch]).
struct B2GemmF32Args {
  const float* x;
  const float* w;
  float* y;
  const float* gate;
  int64_t ldx, ldw, ldy, ld_gate;
  float cap;
  int32_t M, N, K, batch, epilogue, gate_heads;
};
int b2_gemm_f32(const B2GemmF32Args* a, cudaStream_t stream);
// Gated linear unit (B2EpiAct) of rows whose gate and up columns alternate in blocks of 16.
int b2_glu_f32(const float* gate_up, float* out, int64_t rows, int ffn, const struct B2EpiAct* act, cudaStream_t stream);
int b2_gather_rows_f32(const float* src, const int64_t* index, float* out, int rows_out, int cols, int64_t rows_src,
                       b2::Status* status, cudaStream_t stream);
// Causal GQA attention over the paged cache in f32: any head sizes up to 1024, decode rows and prompt chunks alike. Row t
// of sequence row_seq[t] sees positions 0 .. positions[t]. Keys are `dim` columns apart, values (the first vdim of) ld_v, rows of
// out ld_out. gate, gate_elems and mods as in b2/api.h, the gate f32.
int b2_attn_f32(const float* q, const float* k_cache, const float* v_cache, float* out, const int32_t* row_seq,
                const int32_t* positions, const int32_t* block_tables, int rows, int seqs, int max_blocks, int n_q, int n_kv,
                int dim, int vdim, int64_t ld_v, int64_t ld_out, int page_size, float scale, const struct B2AttnMods* mods,
                int64_t num_pages, const float* gate, int64_t gate_stride, int gate_elems, b2::Status* status, cudaStream_t stream);

#ifdef __cplusplus
}
#endif
