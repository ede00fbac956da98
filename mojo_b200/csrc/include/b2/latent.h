// C launch API around latent attention (one cached vector per token, from which every head's key and value are linear
// maps), products with one small weight per head, and mixture-of-experts layers whose experts all live on this GPU.
// Conventions as in b2/mixers.h; the attention itself is b2_latent_attend_bf16 in b2/api.h.
#pragma once
#include <cstdint>
#include <cuda_runtime.h>
#include "b2/api.h"
#include "b2/status.h"

#ifdef __cplusplus
extern "C" {
#endif

// cache[slots[t], 0:rank] = rms_norm(c[t, 0:rank]) * weight, columns rank .. pad - 1 zero; slots < 0 are skipped.
int b2_latent_write(const void* c, int64_t ld, const float* weight, float eps, const int64_t* slots, void* cache, int rows, int rank, int pad,
                    int64_t num_slots, int f32, b2::Status* status, cudaStream_t stream);
// Latent attention with rotary positions, neighbouring columns in pairs: the same for the latent, and the shared key part
// k [rows, rot] (row stride ld) rotated into cache columns column .. column + rot; other columns up to `pad` become zero. The
// queries q [rows, heads * q_dim] (row stride ld_q) rotate in place, columns q_off .. q_off + rot of each head.
// cos_sin f32 [max_pos, rot]: cosines, then sines.
struct B2LatentRopeArgs {
  const void* c;
  const void* k;
  void* q;
  const float* weight;
  const int64_t* slots;
  void* cache;
  const float* cos_sin;
  const int32_t* positions;
  int64_t ld, ld_q, num_slots;
  float eps;
  int32_t rows, rank, rot, column, pad, heads, q_dim, q_off, max_pos;
};
int b2_latent_write_rope(const struct B2LatentRopeArgs* a, int f32, b2::Status* status, cudaStream_t stream);
// Copies the latents of whole contexts out of their cache pages: scratch page p (128 rows) holds positions
// 128 * pages[p][1] ... of sequence pages[p][0]; rows past the sequence's context are zero.
int b2_latent_gather_bf16(const void* cache, const int32_t* pages, const int32_t* ctx_lens, const int32_t* block_tables, void* out, int n_pages,
                          int seqs, int max_blocks, int page_size, int pad, int64_t num_pages, b2::Status* status, cudaStream_t stream);
// y[t, h * n + j] = sum_k x[t, h * k_dim + k] w[h * n + j, k], times sigmoid(gate[t, h * n + j]) where a gate is given, or
// sigmoid(gate[t, h]) with `gate_heads`. k_dim and n multiples of 64.
int b2_head_gemm_bf16(const void* x, const void* w, void* y, const void* gate, int rows, int heads, int n, int k_dim, int64_t ldx, int64_t ldw, int64_t ldy,
                      int64_t ld_gate, int gate_heads, b2::Status* status, cudaStream_t stream);

// Router: scores of `experts + identity` f32 logits per row (0: softmax, 1: sigmoid), the `top` largest (lowest index on ties),
// their scores (divided by their sum with `norm_top`) times `scale`. `correction` (may be null) is added to the scores for the
// choice alone; with keep < groups the choice is among the `keep` groups of neighbours with the largest scores in them. Writes
// weights and ids [rows, top], the place of every (row, choice) among those of its expert, and adds to counts [experts] (zero
// on entry; ids from `experts` on are not counted).
int b2_moe_route(const float* logits, int64_t ld, const float* correction, float* weights, int32_t* ids, int32_t* place, int32_t* counts, int rows,
                 int experts, int identity, int top, int groups, int keep, int scoring, int norm_top, float scale, cudaStream_t stream);
// Rows sorted by expert: xs[slot[t, j]] = x[t], times weights[t, j] where `weights` (may be null) is given (ids from `experts` on get slot -1 and no row). Also lists the tiles of at most `bn` rows of one expert as
// {expert, first row, rows, 0} in tiles (room for experts + rows * top / bn entries), their number in n_tiles[0], and
// leaves counts (and the ticket word counts[experts]) at zero.
int b2_moe_gather(const void* x, const int32_t* ids, const int32_t* place, const float* weights, int32_t* counts, int32_t* slot, void* xs, int32_t* tiles, int32_t* n_tiles,
                  int rows, int experts, int top, int width, int bn, int f32, b2::Status* status, cudaStream_t stream);
// y[r] = x[r] W[e]^T for the rows of every listed tile; w [experts, n, k]. `epilogue` NONE, RELU2 or SWIGLU (gate and up rows
// interleaved in blocks of 16, y then has n / 2 columns).
int b2_moe_tiles_gemm_bf16(const void* x, const void* w, const int32_t* tiles, const int32_t* n_tiles, void* y, int rows, int experts, int n, int k,
                           int epilogue, const struct B2EpiAct* act, int bn, b2::Status* status, cudaStream_t stream);
// The same product in true f32 (epilogue NONE or RELU2), for tiles of at most 64 rows.
int b2_moe_tiles_gemm_f32(const float* x, const float* w, const int32_t* tiles, const int32_t* n_tiles, float* y, int max_tiles, int n, int k,
                          int epilogue, cudaStream_t stream);

#ifdef __cplusplus
}
#endif
