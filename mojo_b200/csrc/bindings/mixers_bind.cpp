// Bindings of the sequence-mixing kernels (b2/mixers.h): argument checks, then raw pointers on the current stream.
#include <torch/extension.h>
#include <c10/cuda/CUDAStream.h>
#include <c10/cuda/CUDAGuard.h>
#include "b2/launch.h"
#include "b2/mixers.h"

namespace py = pybind11;

namespace {
using OptTensor = c10::optional<at::Tensor>;

cudaStream_t cur_stream() { return c10::cuda::getCurrentCUDAStream().stream(); }
void check(int rc, const char* what) {
  if (rc == 0) return;
  if (b2::is_cuda_rc(rc)) {
    const cudaError_t e = b2::cuda_error_of(rc);
    throw std::runtime_error(std::string("mojo_b200: ") + what + " failed: CUDA error " + std::to_string(static_cast<int>(e)) + " (" +
                             cudaGetErrorName(e) + ": " + cudaGetErrorString(e) + ")");
  }
  throw std::runtime_error(std::string("mojo_b200: ") + what + " rejected its arguments: " + b2::status_code_name(-rc));
}
void need(bool cond, const char* msg) {
  if (!cond) throw std::invalid_argument(std::string("mojo_b200: ") + msg);
}
b2::Status* status_ptr(const OptTensor& s) { return s.has_value() ? reinterpret_cast<b2::Status*>(s->data_ptr()) : nullptr; }
bool is_act(const at::Tensor& t) { return t.is_cuda() && (t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat); }
bool is_f32(const at::Tensor& t, int64_t n) { return t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() == n; }
bool is_i32(const at::Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous(); }
bool is_i64(const at::Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kLong && t.is_contiguous(); }
template <typename P>
P* opt(const OptTensor& t) { return t.has_value() ? static_cast<P*>(t->data_ptr()) : nullptr; }

B2SeqRows seq_rows_of(const at::Tensor& row_seq, const at::Tensor& seq_rows, const at::Tensor& seq_state, int64_t banks) {
  need(is_i32(row_seq) && is_i32(seq_rows) && is_i32(seq_state) && seq_rows.numel() == seq_state.numel() && seq_rows.numel() % 2 == 0,
       "sequence rows: int32 row_seq [T], seq_rows [S, 2], seq_state [S, 2]");
  B2SeqRows s{};
  s.row_seq = row_seq.data_ptr<int32_t>();
  s.seq_rows = seq_rows.data_ptr<int32_t>();
  s.seq_state = seq_state.data_ptr<int32_t>();
  s.rows = static_cast<int32_t>(row_seq.numel());
  s.seqs = static_cast<int32_t>(seq_rows.numel() / 2);
  s.banks = static_cast<int32_t>(banks);
  return s;
}

void hyper_norm(at::Tensor& x, const OptTensor& y, const OptTensor& mix, const OptTensor& out, const OptTensor& in, const at::Tensor& weight,
                at::Tensor& h, const OptTensor& ids, const OptTensor& embed, double embed_scale, const OptTensor& rows_index, bool store, double eps,
                int64_t mean_width, const OptTensor& status) {
  need(x.dim() == 3 && x.is_cuda() && x.scalar_type() == at::kFloat && x.is_contiguous(), "hyper_norm: x must be contiguous CUDA f32 [rows, streams, width]");
  const int64_t T = x.size(0), S = x.size(1), W = x.size(2);
  need(is_act(h) && h.dim() == 2 && h.is_contiguous() && h.size(1) == W && is_f32(weight, W), "hyper_norm: h [n, width], weight f32 [width]");
  if (y.has_value()) {
    need(y->scalar_type() == h.scalar_type() && y->is_contiguous() && y->numel() == T * W, "hyper_norm: y [rows, width] like h");
    need(mix.has_value() && out.has_value() && is_f32(*mix, S * S) && is_f32(*out, S), "hyper_norm: mix [S, S] and out [S] f32");
  }
  if (in.has_value()) need(is_f32(*in, S), "hyper_norm: in f32 [S]");
  if (ids.has_value())
    need(is_i64(*ids) && ids->numel() == T && embed.has_value() && embed->scalar_type() == h.scalar_type() && embed->is_contiguous() && embed->size(1) == W,
         "hyper_norm: ids int64 [rows], embed [vocab, width] like h");
  if (rows_index.has_value()) need(is_i64(*rows_index) && rows_index->numel() == h.size(0), "hyper_norm: rows_index int64 [n]");
  else need(h.size(0) == T, "hyper_norm: h must have one row per x row");
  B2HyperArgs a{};
  a.x = x.data_ptr<float>();
  a.y = opt<const void>(y);
  a.mix = opt<const float>(mix);
  a.out = opt<const float>(out);
  a.in = opt<const float>(in);
  a.weight = weight.data_ptr<float>();
  a.h = h.data_ptr();
  a.ids = opt<const int64_t>(ids);
  a.embed = opt<const void>(embed);
  a.rows_index = opt<const int64_t>(rows_index);
  a.embed_scale = static_cast<float>(embed_scale);
  a.eps = static_cast<float>(eps);
  a.n_out = static_cast<int32_t>(h.size(0));
  a.rows = static_cast<int32_t>(T);
  a.width = static_cast<int32_t>(W);
  a.mean_width = static_cast<int32_t>(mean_width);
  a.streams = static_cast<int32_t>(S);
  a.vocab = embed.has_value() ? static_cast<int32_t>(embed->size(0)) : 0;
  a.store = store ? 1 : 0;
  c10::cuda::CUDAGuard g(x.device());
  check(b2_hyper_norm(&a, h.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "hyper_norm");
}

void conv_qkv(const at::Tensor& proj, const at::Tensor& conv_w, const OptTensor& conv_state, const at::Tensor& cos_sin, const at::Tensor& positions,
              const at::Tensor& row_seq, const at::Tensor& seq_rows, const at::Tensor& seq_state, int64_t banks, at::Tensor& q_out,
              const OptTensor& slots, const OptTensor& k_cache, const OptTensor& v_cache, int64_t heads, int64_t kv_heads, int64_t dim, int64_t vdim,
              double eps, const OptTensor& status) {
  need(is_act(proj) && proj.dim() == 2 && proj.stride(1) == 1, "conv_qkv: proj must be 2-D with unit inner stride");
  const int64_t T = proj.size(0), taps = conv_w.size(0), channels = heads * dim + kv_heads * (dim + vdim);
  need(conv_w.dim() == 2 && is_f32(conv_w, taps * channels) && proj.size(1) >= channels, "conv_qkv: conv_w f32 [taps, channels], proj at least that wide");
  need(cos_sin.is_cuda() && cos_sin.scalar_type() == at::kFloat && cos_sin.is_contiguous() && cos_sin.dim() == 2, "conv_qkv: cos_sin f32 [max_pos, rot]");
  need(is_i32(positions) && positions.numel() == T && row_seq.numel() == T, "conv_qkv: positions, row_seq int32 [T]");
  need(q_out.scalar_type() == proj.scalar_type() && q_out.is_contiguous() && q_out.size(0) == T && q_out.size(1) % heads == 0, "conv_qkv: q_out [T, heads * pad]");
  const B2SeqRows s = seq_rows_of(row_seq, seq_rows, seq_state, banks);
  B2ConvQkvArgs a{};
  if (taps > 1) need(conv_state.has_value() && conv_state->scalar_type() == proj.scalar_type() && conv_state->is_contiguous() &&
                         conv_state->numel() == banks * (taps - 1) * channels, "conv_qkv: conv_state [banks, taps - 1, channels] like proj");
  if (kv_heads > 0) {
    need(k_cache.has_value() && v_cache.has_value() && slots.has_value() && is_i64(*slots) && slots->numel() == T, "conv_qkv: caches and int64 slots [T]");
    need(k_cache->dim() == 4 && v_cache->dim() == 4 && k_cache->is_contiguous() && v_cache->is_contiguous() && k_cache->scalar_type() == proj.scalar_type() &&
             v_cache->scalar_type() == proj.scalar_type() && k_cache->size(1) == kv_heads && v_cache->size(1) == kv_heads &&
             k_cache->size(0) == v_cache->size(0) && k_cache->size(2) == v_cache->size(2),
         "conv_qkv: caches [pages, kv_heads, page, pad] like proj");
    a.page_size = static_cast<int32_t>(k_cache->size(2));
    a.num_slots = k_cache->size(0) * k_cache->size(2);
    a.pad_vdim = static_cast<int32_t>(v_cache->size(3));
    need(k_cache->size(3) == q_out.size(1) / heads, "conv_qkv: queries and keys must be padded alike");
  }
  a.proj = proj.data_ptr();
  a.ld = proj.stride(0);
  a.conv_w = conv_w.data_ptr<float>();
  a.conv_state = opt<void>(conv_state);
  a.cos_sin = cos_sin.data_ptr<float>();
  a.positions = positions.data_ptr<int32_t>();
  a.slots = opt<const int64_t>(slots);
  a.q_out = q_out.data_ptr();
  a.k_cache = opt<void>(k_cache);
  a.v_cache = opt<void>(v_cache);
  a.heads = static_cast<int32_t>(heads);
  a.kv_heads = static_cast<int32_t>(kv_heads);
  a.dim = static_cast<int32_t>(dim);
  a.vdim = static_cast<int32_t>(vdim);
  a.pad_dim = static_cast<int32_t>(q_out.size(1) / heads);
  a.rot = static_cast<int32_t>(cos_sin.size(1));
  a.taps = static_cast<int32_t>(taps);
  a.max_pos = static_cast<int32_t>(cos_sin.size(0));
  a.eps = static_cast<float>(eps);
  c10::cuda::CUDAGuard g(proj.device());
  check(b2_conv_qkv(&a, &s, proj.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "conv_qkv");
}

void delta_rule(const at::Tensor& proj, const at::Tensor& decay, const at::Tensor& gate, bool gate_silu, const at::Tensor& conv_w, const OptTensor& conv_state, const at::Tensor& neg_rate,
                const at::Tensor& dt_bias, const at::Tensor& norm_w, at::Tensor& state, const at::Tensor& row_seq, const at::Tensor& seq_rows,
                const at::Tensor& seq_state, at::Tensor& out, const at::Tensor& scratch, const OptTensor& o_raw, int64_t b_off, int64_t heads,
                int64_t kv_heads, int64_t dim, int64_t vdim, double eps, int64_t n_decode, int64_t first, int64_t n_prefill, const OptTensor& status) {
  need(is_act(proj) && proj.dim() == 2 && proj.stride(1) == 1 && decay.scalar_type() == proj.scalar_type() && decay.dim() == 2 && decay.stride(1) == 1 &&
           gate.scalar_type() == proj.scalar_type() && gate.dim() == 2 && gate.stride(1) == 1 && out.scalar_type() == proj.scalar_type() && out.dim() == 2 && out.stride(1) == 1, "delta_rule: proj, decay, gate, out of one type with unit inner strides");
  const int64_t T = proj.size(0), taps = conv_w.size(0), channels = 2 * kv_heads * dim + heads * vdim;
  const bool head_decay = dt_bias.numel() == heads && dim != 1;
  need(decay.size(0) == T && decay.size(1) >= heads * (head_decay ? 1 : dim) && gate.size(0) == T && gate.size(1) >= heads * vdim && out.size(0) == T && out.size(1) >= heads * vdim && proj.size(1) >= channels && b_off >= 0 &&
           b_off + heads <= proj.size(1) && row_seq.numel() == T, "delta_rule: shape mismatch");
  need(conv_w.dim() == 2 && is_f32(conv_w, taps * channels) && is_f32(neg_rate, heads) && is_f32(dt_bias, heads * (head_decay ? 1 : dim)) && is_f32(norm_w, vdim),
       "delta_rule: f32 parameters");
  need(state.dim() == 4 && state.is_cuda() && state.scalar_type() == at::kFloat && state.is_contiguous() && state.size(1) == heads && state.size(2) == dim &&
           state.size(3) == vdim, "delta_rule: state f32 [slots, heads, dim, vdim]");
  const int64_t banks = 2 * state.size(0);
  if (taps > 1) need(conv_state.has_value() && conv_state->scalar_type() == proj.scalar_type() && conv_state->is_contiguous() &&
                         conv_state->numel() == banks * (taps - 1) * channels, "delta_rule: conv_state [banks, taps - 1, channels] like proj");
  const B2SeqRows s = seq_rows_of(row_seq, seq_rows, seq_state, banks);
  B2DeltaArgs a{};
  a.proj = proj.data_ptr();
  a.decay = decay.data_ptr();
  a.gate = gate.data_ptr();
  a.ld = proj.stride(0);
  a.ld_decay = decay.stride(0);
  a.ld_gate = gate.stride(0);
  a.head_decay = head_decay ? 1 : 0;
  a.gate_silu = gate_silu ? 1 : 0;
  a.conv_w = conv_w.data_ptr<float>();
  a.conv_state = opt<void>(conv_state);
  a.neg_rate = neg_rate.data_ptr<float>();
  a.dt_bias = dt_bias.data_ptr<float>();
  a.norm_w = norm_w.data_ptr<float>();
  a.state = state.data_ptr<float>();
  a.out = out.data_ptr();
  a.ld_out = out.stride(0);
  a.b_off = static_cast<int32_t>(b_off);
  a.heads = static_cast<int32_t>(heads);
  a.kv_heads = static_cast<int32_t>(kv_heads);
  a.dim = static_cast<int32_t>(dim);
  a.vdim = static_cast<int32_t>(vdim);
  a.taps = static_cast<int32_t>(taps);
  a.eps = static_cast<float>(eps);
  const int f32 = proj.scalar_type() == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard g(proj.device());
  need(is_f32(scratch, b2_delta_scratch_floats(a.heads, a.dim, a.vdim, s.rows, s.seqs)), "delta_rule: f32 scratch of delta_scratch_floats elements");
  a.scratch = scratch.data_ptr<float>();
  if (o_raw.has_value()) {
    need(is_f32(*o_raw, T * heads * vdim), "delta_rule: o_raw f32 [T, heads * vdim]");
    a.o_raw = o_raw->data_ptr<float>();
  }
  check(b2_delta_rule(&a, &s, static_cast<int>(n_decode), static_cast<int>(first), static_cast<int>(n_prefill), f32, status_ptr(status), cur_stream()),
        "delta_rule");
}

void gemm_f32(const at::Tensor& x, const at::Tensor& w, at::Tensor& y, int64_t batch, int64_t epilogue, double cap, const OptTensor& gate) {
  for (const at::Tensor* t : {&x, &w, static_cast<const at::Tensor*>(&y)})
    need(t->is_cuda() && t->scalar_type() == at::kFloat && t->dim() == 2 && t->stride(1) == 1, "gemm_f32: 2-D CUDA f32 with unit inner strides");
  const int64_t K = w.size(1);
  need(batch >= 1 && w.size(0) % batch == 0 && x.size(1) == batch * K && y.size(0) == x.size(0) && y.size(1) == w.size(0),
       "gemm_f32: x [M, batch * K], w [batch * N, K], y [M, batch * N]");
  B2GemmF32Args a{};
  if (gate.has_value()) {
    need(gate->is_cuda() && gate->scalar_type() == at::kFloat && gate->dim() == 2 && gate->stride(1) == 1 && gate->size(0) == y.size(0) &&
             (gate->size(1) == y.size(1) || gate->size(1) == batch), "gemm_f32: gate f32 like y, or one column per product");
    a.gate_heads = gate->size(1) == y.size(1) ? 0 : 1;
  }
  a.x = x.data_ptr<float>();
  a.w = w.data_ptr<float>();
  a.y = y.data_ptr<float>();
  a.gate = opt<const float>(gate);
  a.ldx = x.stride(0);
  a.ldw = w.stride(0);
  a.ldy = y.stride(0);
  a.ld_gate = gate.has_value() ? gate->stride(0) : 0;
  a.cap = static_cast<float>(cap);
  a.M = static_cast<int32_t>(x.size(0));
  a.N = static_cast<int32_t>(w.size(0) / batch);
  a.K = static_cast<int32_t>(K);
  a.batch = static_cast<int32_t>(batch);
  a.epilogue = static_cast<int32_t>(epilogue);
  c10::cuda::CUDAGuard g(x.device());
  check(b2_gemm_f32(&a, cur_stream()), "gemm_f32");
}

void residual_norm(at::Tensor& x, const OptTensor& y, const OptTensor& experts, const OptTensor& slot, const OptTensor& expert_w, const OptTensor& y_scale,
                   const OptTensor& weight, at::Tensor& h, const OptTensor& ids, const OptTensor& embed, double embed_scale, const OptTensor& prev,
                   const OptTensor& bigram, int64_t mul_prev, int64_t mul_cur, const OptTensor& x0, const OptTensor& rows_index, bool store, double eps,
                   int64_t mean_width, const OptTensor& status, const OptTensor& bias, const OptTensor& own, const OptTensor& gated,
                   const OptTensor& gate) {
  need(x.dim() == 2 && x.is_cuda() && x.scalar_type() == at::kFloat && x.is_contiguous(), "residual_norm: x must be contiguous CUDA f32 [rows, width]");
  const int64_t T = x.size(0), W = x.size(1);
  need(is_act(h) && h.dim() == 2 && h.stride(1) == 1 && h.size(1) == W, "residual_norm: h [n, width]");
  B2ResidualArgs a{};
  if (y.has_value()) need(y->scalar_type() == h.scalar_type() && y->is_contiguous() && y->numel() == T * W, "residual_norm: y [rows, width] like h");
  if (y_scale.has_value()) need(is_f32(*y_scale, W), "residual_norm: y_scale f32 [width]");
  if (bias.has_value()) need(weight.has_value() && is_f32(*bias, W), "residual_norm: bias f32 [width] beside a weight");
  for (const OptTensor* t : {&own, &gated})
    if (t->has_value()) need((*t)->scalar_type() == h.scalar_type() && (*t)->is_contiguous() && (*t)->numel() == T * W, "residual_norm: own, gated [rows, width] like h");
  if (gated.has_value()) {
    need(gate.has_value() && gate->is_cuda() && gate->scalar_type() == at::kFloat && gate->dim() == 1 && gate->size(0) == T, "residual_norm: gate f32 [rows]");
    a.ld_gate = gate->stride(0);
  }
  if (weight.has_value()) need(is_f32(*weight, W), "residual_norm: weight f32 [width]");
  if (experts.has_value()) {
    need(experts->scalar_type() == h.scalar_type() && experts->dim() == 2 && experts->is_contiguous() && experts->size(1) == W && slot.has_value() &&
             is_i32(*slot) && slot->dim() == 2 && slot->size(0) == T && (!expert_w.has_value() || is_f32(*expert_w, slot->numel())),
         "residual_norm: expert rows [n, width] like h, slots int32 and weights f32 [rows, top]");
    a.top = static_cast<int32_t>(slot->size(1));
    a.expert_rows = static_cast<int32_t>(experts->size(0));
  }
  if (ids.has_value())
    need(is_i64(*ids) && ids->numel() == T && embed.has_value() && embed->scalar_type() == h.scalar_type() && embed->is_contiguous() && embed->size(1) == W,
         "residual_norm: ids int64 [rows], embed [vocab, width] like h");
  if (bigram.has_value()) {
    need(ids.has_value() && prev.has_value() && is_i32(*prev) && prev->numel() == T && bigram->scalar_type() == h.scalar_type() && bigram->is_contiguous() &&
             bigram->dim() == 2 && bigram->size(1) == W && bigram->size(0) >= 2, "residual_norm: prev int32 [rows], bigram [buckets + 1, width] like h");
    a.buckets = bigram->size(0) - 1;
  }
  if (x0.has_value()) {
    need(x0->scalar_type() == h.scalar_type() && x0->dim() == 2 && x0->stride(1) == 1 && x0->size(0) == T && x0->size(1) == W, "residual_norm: x0 [rows, width] like h");
    a.ld_x0 = x0->stride(0);
  }
  if (rows_index.has_value()) need(is_i64(*rows_index) && rows_index->numel() == h.size(0), "residual_norm: rows_index int64 [n]");
  else need(h.size(0) == T, "residual_norm: h must have one row per x row");
  a.x = x.data_ptr<float>();
  a.y = opt<const void>(y);
  a.experts = opt<const void>(experts);
  a.expert_slot = opt<const int32_t>(slot);
  a.expert_w = opt<const float>(expert_w);
  a.y_scale = opt<const float>(y_scale);
  a.weight = opt<const float>(weight);
  a.h = h.data_ptr();
  a.ids = opt<const int64_t>(ids);
  a.embed = opt<const void>(embed);
  a.prev = opt<const int32_t>(prev);
  a.bigram = opt<const void>(bigram);
  a.x0 = opt<void>(x0);
  a.rows_index = opt<const int64_t>(rows_index);
  a.bias = opt<const float>(bias);
  a.own = opt<const void>(own);
  a.gated = opt<const void>(gated);
  a.gate = gated.has_value() ? opt<const float>(gate) : nullptr;
  a.ld_h = h.stride(0);
  a.mul_prev = mul_prev;
  a.mul_cur = mul_cur;
  a.embed_scale = static_cast<float>(embed_scale);
  a.eps = static_cast<float>(eps);
  a.n_out = static_cast<int32_t>(h.size(0));
  a.rows = static_cast<int32_t>(T);
  a.width = static_cast<int32_t>(W);
  a.mean_width = static_cast<int32_t>(mean_width);
  a.vocab = embed.has_value() ? static_cast<int32_t>(embed->size(0)) : 0;
  a.store = store ? 1 : 0;
  c10::cuda::CUDAGuard g(x.device());
  check(b2_residual_norm(&a, h.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "residual_norm");
}

void attn_f32(const at::Tensor& q, const at::Tensor& k_cache, const at::Tensor& v_cache, at::Tensor& out, const at::Tensor& row_seq,
              const at::Tensor& positions, const at::Tensor& block_tables, double scale, const OptTensor& gate, const OptTensor& status, int64_t window,
              double softcap, double out_scale, int64_t chunk, bool sink, const OptTensor& distance) {
  need(q.is_cuda() && q.scalar_type() == at::kFloat && q.dim() == 2 && q.is_contiguous() && out.scalar_type() == at::kFloat && out.dim() == 2 &&
           out.stride(1) == 1, "attn_f32: q contiguous CUDA f32, out f32 with unit inner stride");
  // values: a cache like the keys', or the first columns of one
  need(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.is_contiguous() && k_cache.scalar_type() == at::kFloat && v_cache.scalar_type() == at::kFloat &&
           k_cache.size(0) == v_cache.size(0) && k_cache.size(1) == v_cache.size(1) && k_cache.size(2) == v_cache.size(2) && v_cache.stride(3) == 1 &&
           v_cache.stride(1) == v_cache.size(2) * v_cache.stride(2) && v_cache.stride(0) == v_cache.size(1) * v_cache.stride(1),
       "attn_f32: f32 caches [pages, n_kv, page, D]");
  const int64_t T = q.size(0), D = k_cache.size(3), n_q = q.size(1) / D;
  need(n_q * D == q.size(1) && out.size(0) == T && out.size(1) == n_q * v_cache.size(3), "attn_f32: shape mismatch");
  need(is_i32(row_seq) && is_i32(positions) && is_i32(block_tables) && row_seq.numel() >= T && positions.numel() >= T && block_tables.dim() == 2, "attn_f32: int32 metadata");
  if (gate.has_value()) need(gate->scalar_type() == at::kFloat && gate->dim() == 2 && gate->size(0) == T && (gate->size(1) == n_q || gate->size(1) == out.size(1)) && gate->stride(1) == 1, "attn_f32: gate f32 [T, n_q], or like out");
  B2AttnMods mods{static_cast<int32_t>(window), static_cast<int32_t>(chunk), static_cast<float>(softcap), static_cast<float>(out_scale), nullptr, sink ? 1 : 0};
  if (distance.has_value()) {
    need(is_f32(*distance, 2 * n_q), "attn_f32: distance f32 [2, n_q]");
    mods.distance = distance->data_ptr<float>();
  }
  c10::cuda::CUDAGuard g(q.device());
  check(b2_attn_f32(q.data_ptr<float>(), k_cache.data_ptr<float>(), v_cache.data_ptr<float>(), out.data_ptr<float>(), row_seq.data_ptr<int32_t>(),
                    positions.data_ptr<int32_t>(), block_tables.data_ptr<int32_t>(), static_cast<int>(T), static_cast<int>(block_tables.size(0)),
                    static_cast<int>(block_tables.size(1)), static_cast<int>(n_q), static_cast<int>(k_cache.size(1)), static_cast<int>(D),
                    static_cast<int>(v_cache.size(3)), v_cache.stride(2), out.stride(0), static_cast<int>(k_cache.size(2)), static_cast<float>(scale),
                    &mods, k_cache.size(0),
                    gate.has_value() ? gate->data_ptr<float>() : nullptr, gate.has_value() ? gate->stride(0) : 0, gate.has_value() && gate->size(1) != n_q ? 1 : 0, status_ptr(status), cur_stream()),
        "attn_f32");
}

void norm_qkv(const at::Tensor& proj, const at::Tensor& bias, const at::Tensor& q_norm, const at::Tensor& k_norm, const at::Tensor& cos_sin,
              const at::Tensor& positions, const at::Tensor& slots, at::Tensor& k_cache, at::Tensor& v_cache, at::Tensor& q_out, int64_t heads,
              int64_t kv_heads, int64_t dim, int64_t vdim, double eps, const OptTensor& status) {
  need(is_act(proj) && proj.dim() == 2 && proj.stride(1) == 1, "norm_qkv: proj must be 2-D with unit inner stride");
  const int64_t T = proj.size(0), channels = heads * dim + kv_heads * (dim + vdim);
  need(proj.size(1) >= channels && is_f32(bias, channels) && is_f32(q_norm, heads * dim) && is_f32(k_norm, kv_heads * dim), "norm_qkv: f32 parameters, proj as wide");
  need(cos_sin.is_cuda() && cos_sin.scalar_type() == at::kFloat && cos_sin.is_contiguous() && cos_sin.dim() == 2, "norm_qkv: cos_sin f32 [max_pos, rot]");
  need(is_i32(positions) && positions.numel() == T && is_i64(slots) && slots.numel() == T, "norm_qkv: positions int32 [T], slots int64 [T]");
  need(q_out.scalar_type() == proj.scalar_type() && q_out.is_contiguous() && q_out.size(0) == T && q_out.size(1) % heads == 0, "norm_qkv: q_out [T, heads * pad]");
  need(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() && k_cache.scalar_type() == proj.scalar_type() &&
           v_cache.scalar_type() == proj.scalar_type() && k_cache.size(1) == kv_heads && v_cache.size(1) == kv_heads &&
           k_cache.size(0) == v_cache.size(0) && k_cache.size(2) == v_cache.size(2) && k_cache.size(3) == q_out.size(1) / heads,
       "norm_qkv: caches [pages, kv_heads, page, pad] like proj, keys padded like the queries");
  B2NormQkvArgs a{};
  a.proj = proj.data_ptr();
  a.ld = proj.stride(0);
  a.bias = bias.data_ptr<float>();
  a.q_norm = q_norm.data_ptr<float>();
  a.k_norm = k_norm.data_ptr<float>();
  a.cos_sin = cos_sin.data_ptr<float>();
  a.positions = positions.data_ptr<int32_t>();
  a.slots = slots.data_ptr<int64_t>();
  a.q_out = q_out.data_ptr();
  a.k_cache = k_cache.data_ptr();
  a.v_cache = v_cache.data_ptr();
  a.num_slots = k_cache.size(0) * k_cache.size(2);
  a.rows = static_cast<int32_t>(T);
  a.heads = static_cast<int32_t>(heads);
  a.kv_heads = static_cast<int32_t>(kv_heads);
  a.dim = static_cast<int32_t>(dim);
  a.vdim = static_cast<int32_t>(vdim);
  a.pad_dim = static_cast<int32_t>(k_cache.size(3));
  a.pad_vdim = static_cast<int32_t>(v_cache.size(3));
  a.rot = static_cast<int32_t>(cos_sin.size(1));
  a.page_size = static_cast<int32_t>(k_cache.size(2));
  a.max_pos = static_cast<int32_t>(cos_sin.size(0));
  a.eps = static_cast<float>(eps);
  c10::cuda::CUDAGuard g(proj.device());
  check(b2_norm_qkv(&a, proj.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "norm_qkv");
}

void gated_linear(const at::Tensor& proj, const at::Tensor& z, const at::Tensor& decay_bias, const at::Tensor& norm_w, double tau, at::Tensor& state,
                  const at::Tensor& row_seq, const at::Tensor& seq_rows, const at::Tensor& seq_state, at::Tensor& out, const at::Tensor& scratch, int64_t heads,
                  int64_t dim, int64_t vdim, double eps, double out_scale, int64_t n_decode, int64_t first, int64_t n_prefill, const OptTensor& status) {
  need(is_act(proj) && proj.dim() == 2 && proj.stride(1) == 1 && out.scalar_type() == proj.scalar_type() && out.dim() == 2 && out.stride(1) == 1 &&
           z.is_cuda() && z.scalar_type() == at::kFloat && z.dim() == 2 && z.stride(1) == 1, "gated_linear: proj and out of one type, z f32, unit inner strides");
  const int64_t T = proj.size(0);
  need(proj.size(1) == 2 * heads * (dim + vdim) && z.size(0) == T && z.size(1) >= heads * dim && out.size(0) == T && out.size(1) == heads * vdim &&
           row_seq.numel() == T && tau > 0.0, "gated_linear: shape mismatch");
  need(is_f32(decay_bias, heads * dim) && is_f32(norm_w, vdim), "gated_linear: f32 parameters");
  need(state.dim() == 4 && state.is_cuda() && state.scalar_type() == at::kFloat && state.is_contiguous() && state.size(1) == heads && state.size(2) == dim &&
           state.size(3) == vdim, "gated_linear: state f32 [slots, heads, dim, vdim]");
  const B2SeqRows s = seq_rows_of(row_seq, seq_rows, seq_state, 2 * state.size(0));
  B2GatedLinearArgs a{};
  a.proj = proj.data_ptr();
  a.z = z.data_ptr<float>();
  a.ld = proj.stride(0);
  a.ld_z = z.stride(0);
  a.decay_bias = decay_bias.data_ptr<float>();
  a.norm_w = norm_w.data_ptr<float>();
  a.state = state.data_ptr<float>();
  a.out = out.data_ptr();
  a.ld_out = out.stride(0);
  a.heads = static_cast<int32_t>(heads);
  a.dim = static_cast<int32_t>(dim);
  a.vdim = static_cast<int32_t>(vdim);
  a.inv_tau = static_cast<float>(1.0 / tau);
  a.eps = static_cast<float>(eps);
  a.out_scale = static_cast<float>(out_scale);
  if (n_prefill > 0) {
    need(is_f32(scratch, b2_gated_linear_scratch_floats(a.heads, a.dim, a.vdim, s.rows, s.seqs, static_cast<int>(n_prefill))), "gated_linear: f32 scratch of gated_linear_scratch_floats elements");
    a.scratch = scratch.data_ptr<float>();
  }
  c10::cuda::CUDAGuard g(proj.device());
  check(b2_gated_linear(&a, &s, static_cast<int>(n_decode), static_cast<int>(first), static_cast<int>(n_prefill), proj.scalar_type() == at::kFloat ? 1 : 0,
                        status_ptr(status), cur_stream()), "gated_linear");
}

void post_norm(const OptTensor& x, const OptTensor& x_out, const OptTensor& y, const OptTensor& experts, const OptTensor& slot, const OptTensor& expert_w,
               const OptTensor& y_scale, double alpha, const OptTensor& weight, const OptTensor& then, const OptTensor& conv_w, const OptTensor& conv_state,
               at::Tensor& h, const OptTensor& ids, const OptTensor& embed, const OptTensor& pos_table, const OptTensor& positions, const OptTensor& rows_index,
               const at::Tensor& row_seq, const at::Tensor& seq_rows, const at::Tensor& seq_state, int64_t banks, int64_t groups, int64_t mean_width, double eps,
               const OptTensor& status) {
  need(is_act(h) && h.dim() == 2 && h.is_contiguous(), "post_norm: h [n, width]");
  const int64_t T = row_seq.numel(), W = h.size(1);
  for (const OptTensor* t : {&x, &x_out})
    if (t->has_value()) need((*t)->dim() == 2 && is_f32(**t, T * W) && (*t)->size(1) == W, "post_norm: x, x_out f32 [rows, width]");
  need(x.has_value() != ids.has_value(), "post_norm: either x or ids");
  for (const OptTensor* t : {&y_scale, &weight, &then})
    if (t->has_value()) need(is_f32(**t, W), "post_norm: y_scale, weight, then f32 [width]");
  if (y.has_value()) need(y->scalar_type() == h.scalar_type() && y->is_contiguous() && y->numel() == T * W, "post_norm: y [rows, width] like h");
  const B2SeqRows s = seq_rows_of(row_seq, seq_rows, seq_state, banks);
  B2PostNormArgs a{};
  if (experts.has_value()) {
    need(experts->scalar_type() == h.scalar_type() && experts->dim() == 2 && experts->is_contiguous() && experts->size(1) == W && slot.has_value() && is_i32(*slot) &&
             slot->dim() == 2 && slot->size(0) == T && (!expert_w.has_value() || is_f32(*expert_w, slot->numel())),
         "post_norm: expert rows [n, width] like h, slots int32 and weights f32 [rows, top]");
    a.top = static_cast<int32_t>(slot->size(1));
    a.expert_rows = static_cast<int32_t>(experts->size(0));
  }
  if (ids.has_value())
    need(is_i64(*ids) && ids->numel() == T && embed.has_value() && embed->scalar_type() == h.scalar_type() && embed->is_contiguous() && embed->dim() == 2 &&
             embed->size(1) == W, "post_norm: ids int64 [rows], embed [vocab, width] like h");
  if (pos_table.has_value()) {
    need(pos_table->scalar_type() == h.scalar_type() && pos_table->is_contiguous() && pos_table->dim() == 2 && pos_table->size(1) == W && positions.has_value() &&
             is_i32(*positions) && positions->numel() == T, "post_norm: pos_table [positions, width] like h, positions int32 [rows]");
    a.max_pos = static_cast<int32_t>(pos_table->size(0));
  }
  if (conv_w.has_value()) {
    a.taps = static_cast<int32_t>(conv_w->size(0));
    need(conv_w->dim() == 2 && is_f32(*conv_w, a.taps * W), "post_norm: conv_w f32 [taps, width]");
    if (a.taps > 1) need(conv_state.has_value() && is_f32(*conv_state, banks * (a.taps - 1) * W), "post_norm: conv_state f32 [banks, taps - 1, width]");
  }
  if (rows_index.has_value()) need(is_i64(*rows_index) && rows_index->numel() == h.size(0), "post_norm: rows_index int64 [n]");
  else need(h.size(0) == T, "post_norm: h must have one row per x row");
  a.x = opt<const float>(x);
  a.x_out = opt<float>(x_out);
  a.y = opt<const void>(y);
  a.experts = opt<const void>(experts);
  a.expert_slot = opt<const int32_t>(slot);
  a.expert_w = opt<const float>(expert_w);
  a.y_scale = opt<const float>(y_scale);
  a.weight = opt<const float>(weight);
  a.then = opt<const float>(then);
  a.conv_w = opt<const float>(conv_w);
  a.conv_state = opt<float>(conv_state);
  a.h = h.data_ptr();
  a.ids = opt<const int64_t>(ids);
  a.embed = opt<const void>(embed);
  a.pos_table = opt<const void>(pos_table);
  a.positions = opt<const int32_t>(positions);
  a.rows_index = opt<const int64_t>(rows_index);
  a.alpha = static_cast<float>(alpha);
  a.eps = static_cast<float>(eps);
  a.n_out = static_cast<int32_t>(h.size(0));
  a.rows = static_cast<int32_t>(T);
  a.width = static_cast<int32_t>(W);
  a.mean_width = static_cast<int32_t>(mean_width);
  a.groups = static_cast<int32_t>(groups);
  a.vocab = embed.has_value() ? static_cast<int32_t>(embed->size(0)) : 0;
  c10::cuda::CUDAGuard g(h.device());
  check(b2_post_norm(&a, &s, h.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "post_norm");
}

void head_norm_qkv(const at::Tensor& proj, const at::Tensor& q_norm, const at::Tensor& k_norm, const at::Tensor& slots, at::Tensor& k_cache, at::Tensor& v_cache,
                   at::Tensor& q_out, int64_t heads, int64_t kv_heads, int64_t vdim, int64_t v_off, double eps, const OptTensor& status) {
  need(is_act(proj) && proj.dim() == 2 && proj.stride(1) == 1, "head_norm_qkv: proj must be 2-D with unit inner stride");
  const int64_t T = proj.size(0), dim = q_norm.numel();
  need(is_f32(q_norm, dim) && is_f32(k_norm, dim) && proj.size(1) >= (heads + kv_heads) * dim && v_off >= 0 && proj.size(1) >= v_off + kv_heads * vdim,
       "head_norm_qkv: f32 weights [dim], proj as wide as its heads");
  need(is_i64(slots) && slots.numel() == T, "head_norm_qkv: slots int64 [T]");
  need(q_out.scalar_type() == proj.scalar_type() && q_out.is_contiguous() && q_out.dim() == 2 && q_out.size(0) == T && q_out.size(1) % heads == 0, "head_norm_qkv: q_out [T, heads * pad]");
  need(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() && k_cache.scalar_type() == proj.scalar_type() &&
           v_cache.scalar_type() == proj.scalar_type() && k_cache.size(1) == kv_heads && v_cache.size(1) == kv_heads && k_cache.size(0) == v_cache.size(0) &&
           k_cache.size(2) == v_cache.size(2) && k_cache.size(3) == q_out.size(1) / heads,
       "head_norm_qkv: caches [pages, kv_heads, page, pad] like proj, keys padded like the queries");
  B2HeadNormArgs a{};
  a.proj = proj.data_ptr();
  a.ld = proj.stride(0);
  a.q_norm = q_norm.data_ptr<float>();
  a.k_norm = k_norm.data_ptr<float>();
  a.slots = slots.data_ptr<int64_t>();
  a.q_out = q_out.data_ptr();
  a.k_cache = k_cache.data_ptr();
  a.v_cache = v_cache.data_ptr();
  a.num_slots = k_cache.size(0) * k_cache.size(2);
  a.rows = static_cast<int32_t>(T);
  a.heads = static_cast<int32_t>(heads);
  a.kv_heads = static_cast<int32_t>(kv_heads);
  a.dim = static_cast<int32_t>(dim);
  a.vdim = static_cast<int32_t>(vdim);
  a.v_off = static_cast<int32_t>(v_off);
  a.pad_dim = static_cast<int32_t>(k_cache.size(3));
  a.pad_vdim = static_cast<int32_t>(v_cache.size(3));
  a.page_size = static_cast<int32_t>(k_cache.size(2));
  a.eps = static_cast<float>(eps);
  c10::cuda::CUDAGuard g(proj.device());
  check(b2_head_norm_qkv(&a, proj.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "head_norm_qkv");
}

void conv_silu(const at::Tensor& proj, const at::Tensor& conv_w, const OptTensor& bias, const OptTensor& conv_state, at::Tensor& out, const at::Tensor& row_seq,
               const at::Tensor& seq_rows, const at::Tensor& seq_state, int64_t banks, const OptTensor& status) {
  need(is_act(proj) && proj.dim() == 2 && proj.stride(1) == 1 && out.scalar_type() == proj.scalar_type() && out.dim() == 2 && out.stride(1) == 1 &&
           out.size(0) == proj.size(0) && row_seq.numel() == proj.size(0), "conv_silu: proj and out of one type with unit inner strides");
  need(conv_w.dim() == 2, "conv_silu: conv_w f32 [taps, channels]");
  const int64_t taps = conv_w.size(0), channels = conv_w.size(1);
  need(is_f32(conv_w, taps * channels) && proj.size(1) >= channels && out.size(1) >= channels && (!bias.has_value() || is_f32(*bias, channels)),
       "conv_silu: f32 parameters, proj and out as wide");
  if (taps > 1) need(conv_state.has_value() && conv_state->scalar_type() == proj.scalar_type() && conv_state->is_contiguous() &&
                         conv_state->numel() == banks * (taps - 1) * channels, "conv_silu: conv_state [banks, taps - 1, channels] like proj");
  const B2SeqRows s = seq_rows_of(row_seq, seq_rows, seq_state, banks);
  B2ConvSiluArgs a{};
  a.proj = proj.data_ptr();
  a.ld = proj.stride(0);
  a.conv_w = conv_w.data_ptr<float>();
  a.bias = opt<const float>(bias);
  a.conv_state = opt<void>(conv_state);
  a.out = out.data_ptr();
  a.ld_out = out.stride(0);
  a.channels = static_cast<int32_t>(channels);
  a.taps = static_cast<int32_t>(taps);
  c10::cuda::CUDAGuard g(proj.device());
  check(b2_conv_silu(&a, &s, proj.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "conv_silu");
}

void selective_scan(const at::Tensor& dt, const at::Tensor& u, const at::Tensor& z, const at::Tensor& b, const at::Tensor& c, const at::Tensor& rate,
                    const at::Tensor& dt_bias, const at::Tensor& d, at::Tensor& state, at::Tensor& out, const at::Tensor& row_seq, const at::Tensor& seq_rows,
                    const at::Tensor& seq_state, int64_t n_decode, int64_t first, int64_t n_prefill, const OptTensor& status) {
  need(state.dim() == 3 && state.is_cuda() && state.scalar_type() == at::kFloat && state.is_contiguous(), "selective_scan: state f32 [slots, channels, states]");
  const int64_t T = row_seq.numel(), ch = state.size(1), n = state.size(2);
  need(dt.is_cuda() && dt.scalar_type() == at::kFloat && dt.dim() == 2 && dt.stride(1) == 1 && dt.size(0) == T && dt.size(1) == ch, "selective_scan: dt f32 [T, channels]");
  for (const at::Tensor* t : {&u, &z, static_cast<const at::Tensor*>(&out)})
    need(is_act(*t) && t->scalar_type() == u.scalar_type() && t->dim() == 2 && t->stride(1) == 1 && t->size(0) == T && t->size(1) == ch, "selective_scan: u, z, out [T, channels]");
  for (const at::Tensor* t : {&b, &c})
    need(t->scalar_type() == u.scalar_type() && t->dim() == 2 && t->stride(1) == 1 && t->size(0) == T && t->size(1) == n && t->stride(0) == b.stride(0), "selective_scan: b, c [T, states]");
  need(is_f32(rate, ch * n) && is_f32(dt_bias, ch) && is_f32(d, ch), "selective_scan: f32 parameters");
  const B2SeqRows s = seq_rows_of(row_seq, seq_rows, seq_state, 2 * state.size(0));
  B2SelectiveScanArgs a{};
  a.dt = dt.data_ptr<float>();
  a.u = u.data_ptr();
  a.z = z.data_ptr();
  a.b = b.data_ptr();
  a.c = c.data_ptr();
  a.ld_dt = dt.stride(0);
  a.ld_u = u.stride(0);
  a.ld_z = z.stride(0);
  a.ld_bc = b.stride(0);
  a.ld_out = out.stride(0);
  a.rate = rate.data_ptr<float>();
  a.dt_bias = dt_bias.data_ptr<float>();
  a.d = d.data_ptr<float>();
  a.state = state.data_ptr<float>();
  a.out = out.data_ptr();
  a.channels = static_cast<int32_t>(ch);
  a.states = static_cast<int32_t>(n);
  c10::cuda::CUDAGuard g(dt.device());
  check(b2_selective_scan(&a, &s, static_cast<int>(n_decode), static_cast<int>(first), static_cast<int>(n_prefill), u.scalar_type() == at::kFloat ? 1 : 0,
                          status_ptr(status), cur_stream()), "selective_scan");
}
}  // namespace

void bind_mixers(py::module_& m) {
  m.def("post_norm", &post_norm, py::arg("x"), py::arg("x_out"), py::arg("y"), py::arg("experts"), py::arg("slot"), py::arg("expert_w"), py::arg("y_scale"),
        py::arg("alpha"), py::arg("weight"), py::arg("then"), py::arg("conv_w"), py::arg("conv_state"), py::arg("h"), py::arg("ids"), py::arg("embed"),
        py::arg("pos_table"), py::arg("positions"), py::arg("rows_index"), py::arg("row_seq"), py::arg("seq_rows"), py::arg("seq_state"), py::arg("banks"),
        py::arg("groups"), py::arg("mean_width"), py::arg("eps"), py::arg("status") = py::none());
  m.def("head_norm_qkv", &head_norm_qkv);
  m.def("conv_silu", &conv_silu);
  m.def("selective_scan", &selective_scan);
  m.def("hyper_norm", &hyper_norm);
  m.def("conv_qkv", &conv_qkv);
  m.def("delta_rule", &delta_rule);
  m.def("delta_scratch_floats", [](int64_t heads, int64_t dim, int64_t vdim, int64_t rows, int64_t seqs) {
    return b2_delta_scratch_floats(static_cast<int>(heads), static_cast<int>(dim), static_cast<int>(vdim), static_cast<int>(rows), static_cast<int>(seqs));
  });
  m.def("norm_qkv", &norm_qkv);
  m.def("gated_linear", &gated_linear);
  m.def("gated_linear_scratch_floats", [](int64_t heads, int64_t dim, int64_t vdim, int64_t rows, int64_t all_seqs, int64_t seqs) {
    return b2_gated_linear_scratch_floats(static_cast<int>(heads), static_cast<int>(dim), static_cast<int>(vdim), static_cast<int>(rows),
                                          static_cast<int>(all_seqs), static_cast<int>(seqs));
  });
  m.def("gated_linear_prefill_launches", [](int64_t heads, int64_t vdim, int64_t rows, int64_t seqs) {
    return b2_gated_linear_prefill_launches(static_cast<int>(heads), static_cast<int>(vdim), static_cast<int>(rows), static_cast<int>(seqs));
  });
  m.def("residual_norm", &residual_norm, py::arg("x"), py::arg("y"), py::arg("experts"), py::arg("slot"), py::arg("expert_w"), py::arg("y_scale"),
        py::arg("weight"), py::arg("h"), py::arg("ids"), py::arg("embed"), py::arg("embed_scale"), py::arg("prev"), py::arg("bigram"), py::arg("mul_prev"),
        py::arg("mul_cur"), py::arg("x0"), py::arg("rows_index"), py::arg("store"), py::arg("eps"), py::arg("mean_width"), py::arg("status") = py::none(),
        py::arg("bias") = py::none(), py::arg("own") = py::none(), py::arg("gated") = py::none(), py::arg("gate") = py::none());
  m.def("gemm_f32", &gemm_f32, py::arg("x"), py::arg("w"), py::arg("y"), py::arg("batch") = 1, py::arg("epilogue") = 0, py::arg("cap") = 0.0,
        py::arg("gate") = py::none());
  m.def("attn_f32", &attn_f32, py::arg("q"), py::arg("k_cache"), py::arg("v_cache"), py::arg("out"), py::arg("row_seq"), py::arg("positions"),
        py::arg("block_tables"), py::arg("scale"), py::arg("gate") = py::none(), py::arg("status") = py::none(), py::arg("window") = 0,
        py::arg("softcap") = 0.0, py::arg("out_scale") = 1.0, py::arg("chunk") = 0, py::arg("sink") = false, py::arg("distance") = py::none());
  m.def("glu_f32", [](const at::Tensor& gu, at::Tensor& out, double limit, double alpha, double up_bias) {
    need(gu.is_cuda() && gu.scalar_type() == at::kFloat && gu.is_contiguous() && out.is_contiguous() && out.scalar_type() == at::kFloat &&
             gu.size(0) == out.size(0) && gu.size(1) == 2 * out.size(1), "glu_f32: gate_up [M, 2F], out [M, F], contiguous CUDA f32");
    const B2EpiAct act{static_cast<float>(limit), static_cast<float>(alpha), static_cast<float>(up_bias), 0.0f};
    c10::cuda::CUDAGuard g(gu.device());
    check(b2_glu_f32(gu.data_ptr<float>(), out.data_ptr<float>(), out.size(0), static_cast<int>(out.size(1)), &act, cur_stream()), "glu_f32");
  });
  m.def("gather_rows_f32", [](const at::Tensor& src, const at::Tensor& index, at::Tensor& out, const OptTensor& status) {
    need(src.is_cuda() && src.scalar_type() == at::kFloat && src.is_contiguous() && src.dim() == 2 && out.is_contiguous() && out.scalar_type() == at::kFloat &&
             is_i64(index) && out.size(0) == index.numel() && out.size(1) == src.size(1), "gather_rows_f32: f32 [rows, cols], int64 index");
    c10::cuda::CUDAGuard g(src.device());
    check(b2_gather_rows_f32(src.data_ptr<float>(), index.data_ptr<int64_t>(), out.data_ptr<float>(), static_cast<int>(index.numel()),
                             static_cast<int>(src.size(1)), src.size(0), status_ptr(status), cur_stream()), "gather_rows_f32");
  });
}
