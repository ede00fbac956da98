// Bindings of latent attention, per-head products and single-GPU mixture-of-experts kernels (b2/latent.h).
#include <array>
#include <torch/extension.h>
#include <c10/cuda/CUDAStream.h>
#include <c10/cuda/CUDAGuard.h>
#include "b2/latent.h"
#include "b2/launch.h"

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
bool is_bf16(const at::Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kBFloat16; }
bool rows_of(const at::Tensor& t) { return t.dim() == 2 && t.stride(1) == 1; }
bool is_f32(const at::Tensor& t, int64_t n) { return t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() == n; }
bool is_i32(const at::Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous(); }
bool is_i64(const at::Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kLong && t.is_contiguous(); }
int as_int(int64_t v) { return static_cast<int>(v); }

void latent_write(const at::Tensor& c, const at::Tensor& weight, double eps, const at::Tensor& slots, at::Tensor& cache, const OptTensor& status,
                  const OptTensor& k, const OptTensor& q, int64_t heads, int64_t q_off, int64_t column, const OptTensor& cos_sin, const OptTensor& positions) {
  need(is_act(c) && rows_of(c) && cache.scalar_type() == c.scalar_type() && cache.is_cuda() && cache.dim() == 3 && cache.is_contiguous(),
       "latent_write: c [T, rank], cache [pages, page, pad] of one type");
  need(is_f32(weight, c.size(1)) && cache.size(2) >= c.size(1) && is_i64(slots) && slots.numel() == c.size(0), "latent_write: weight f32 [rank], slots int64 [T]");
  c10::cuda::CUDAGuard g(c.device());
  if (k.has_value()) {
    need(q.has_value() && cos_sin.has_value() && positions.has_value(), "latent_write: k, q, cos_sin and positions go together");
    const int64_t rot = k->size(1), T = c.size(0);
    need(rows_of(*k) && k->scalar_type() == c.scalar_type() && k->size(0) == T && k->stride(0) == c.stride(0) && rows_of(*q) && q->scalar_type() == c.scalar_type() &&
             q->size(0) == T && heads >= 1 && q->size(1) % heads == 0, "latent_write: k [T, rot] beside c, q [T, heads * q_dim]");
    need(cos_sin->is_cuda() && cos_sin->scalar_type() == at::kFloat && cos_sin->is_contiguous() && cos_sin->dim() == 2 && cos_sin->size(1) == rot && is_i32(*positions) &&
             positions->numel() == T, "latent_write: cos_sin f32 [max_pos, rot], positions int32 [T]");
    B2LatentRopeArgs a{};
    a.c = c.data_ptr();
    a.k = k->data_ptr();
    a.q = q->data_ptr();
    a.weight = weight.data_ptr<float>();
    a.slots = slots.data_ptr<int64_t>();
    a.cache = cache.data_ptr();
    a.cos_sin = cos_sin->data_ptr<float>();
    a.positions = positions->data_ptr<int32_t>();
    a.ld = c.stride(0);
    a.ld_q = q->stride(0);
    a.num_slots = cache.size(0) * cache.size(1);
    a.eps = static_cast<float>(eps);
    a.rows = as_int(T);
    a.rank = as_int(c.size(1));
    a.rot = as_int(rot);
    a.column = as_int(column);
    a.pad = as_int(cache.size(2));
    a.heads = as_int(heads);
    a.q_dim = as_int(q->size(1) / heads);
    a.q_off = as_int(q_off);
    a.max_pos = as_int(cos_sin->size(0));
    check(b2_latent_write_rope(&a, c.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "latent_write");
    return;
  }
  check(b2_latent_write(c.data_ptr(), c.stride(0), weight.data_ptr<float>(), static_cast<float>(eps), slots.data_ptr<int64_t>(), cache.data_ptr(),
                        as_int(c.size(0)), as_int(c.size(1)), as_int(cache.size(2)), cache.size(0) * cache.size(1), c.scalar_type() == at::kFloat ? 1 : 0,
                        status_ptr(status), cur_stream()), "latent_write");
}

void latent_gather(const at::Tensor& cache, const at::Tensor& pages, const at::Tensor& ctx_lens, const at::Tensor& tables, at::Tensor& out,
                   const OptTensor& status) {
  need(is_bf16(cache) && cache.dim() == 3 && cache.is_contiguous() && is_bf16(out) && out.is_contiguous() && out.dim() == 2 && out.size(1) == cache.size(2),
       "latent_gather: cache bf16 [pages, page, pad], out bf16 [rows, pad]");
  need(is_i32(pages) && pages.dim() == 2 && pages.size(1) == 2 && out.size(0) == pages.size(0) * 128 && is_i32(ctx_lens) && is_i32(tables) && tables.dim() == 2 &&
           tables.size(0) == ctx_lens.numel(), "latent_gather: pages int32 [n, 2], 128 rows of out each; int32 metadata");
  c10::cuda::CUDAGuard g(cache.device());
  check(b2_latent_gather_bf16(cache.data_ptr(), pages.data_ptr<int32_t>(), ctx_lens.data_ptr<int32_t>(), tables.data_ptr<int32_t>(), out.data_ptr(),
                              as_int(pages.size(0)), as_int(ctx_lens.numel()), as_int(tables.size(1)), as_int(cache.size(1)), as_int(cache.size(2)),
                              cache.size(0), status_ptr(status), cur_stream()), "latent_gather");
}

void latent_attend(const at::Tensor& q, const at::Tensor& cache, at::Tensor& out, const at::Tensor& row_ctx, const at::Tensor& tables, const OptTensor& row_seq,
                   const OptTensor& workspace, int64_t heads, int64_t splits, double scale, const OptTensor& status, int64_t latent,
                   int64_t window) {
  need(is_bf16(q) && rows_of(q) && is_bf16(cache) && cache.dim() == 3 && cache.is_contiguous() && is_bf16(out) && out.dim() == 2 && out.is_contiguous(),
       "latent_attend: q [R, heads * columns], out [R, heads * latent], cache [pages, page, columns], bf16");
  const int64_t R = q.size(0), D = cache.size(2), L = latent > 0 ? latent : D;
  need(q.size(1) == heads * D && L <= D && out.size(0) == R && out.size(1) == heads * L, "latent_attend: shape mismatch");
  need(is_i32(row_ctx) && row_ctx.numel() >= R && is_i32(tables) && tables.dim() == 2, "latent_attend: int32 metadata");
  if (row_seq.has_value()) need(is_i32(*row_seq) && row_seq->numel() >= R, "latent_attend: row_seq int32 [R]");
  else need(tables.size(0) >= R, "latent_attend: one block table per row when row_seq is not given");
  float* ws = nullptr;
  if (splits > 1) {
    need(workspace.has_value() && workspace->numel() * 4 >= b2_latent_attend_workspace(as_int(R), as_int(heads), as_int(L), as_int(splits)),
         "latent_attend: workspace too small");
    ws = workspace->data_ptr<float>();
  }
  c10::cuda::CUDAGuard g(q.device());
  check(b2_latent_attend_bf16(q.data_ptr(), cache.data_ptr(), out.data_ptr(), row_ctx.data_ptr<int32_t>(), tables.data_ptr<int32_t>(),
                              row_seq.has_value() ? row_seq->data_ptr<int32_t>() : nullptr, ws, as_int(R), as_int(tables.size(1)), as_int(heads), as_int(L),
                              as_int(D - L), as_int(cache.size(1)), as_int(splits), static_cast<float>(scale), as_int(window), cache.size(0), q.stride(0),
                              status_ptr(status), cur_stream()),
        "latent_attend");
}

void token_rows(const at::Tensor& cu_q, const at::Tensor& ctx_lens, at::Tensor& row_ctx, at::Tensor& row_seq) {
  need(is_i32(cu_q) && is_i32(ctx_lens) && cu_q.numel() == ctx_lens.numel() + 1 && is_i32(row_ctx) && is_i32(row_seq), "token_rows: int32 cu_q [S + 1], ctx_lens [S]");
  c10::cuda::CUDAGuard g(cu_q.device());
  check(b2_mla_rows_meta(cu_q.data_ptr<int32_t>(), ctx_lens.data_ptr<int32_t>(), as_int(ctx_lens.numel()), row_ctx.data_ptr<int32_t>(),
                         row_seq.data_ptr<int32_t>(), cur_stream()), "token_rows");
}

void head_gemm(const at::Tensor& x, const at::Tensor& w, at::Tensor& y, int64_t heads, const OptTensor& gate, const OptTensor& status) {
  need(is_bf16(x) && rows_of(x) && is_bf16(w) && rows_of(w) && is_bf16(y) && rows_of(y), "head_gemm: 2-D CUDA bf16");
  need(heads >= 1 && w.size(0) % heads == 0 && x.size(1) == heads * w.size(1) && y.size(0) == x.size(0) && y.size(1) == w.size(0),
       "head_gemm: x [T, heads * K], w [heads * N, K], y [T, heads * N]");
  const bool by_head = gate.has_value() && gate->size(1) != y.size(1);
  if (gate.has_value())
    need(is_bf16(*gate) && rows_of(*gate) && gate->size(0) == y.size(0) && gate->size(1) == (by_head ? heads : y.size(1)), "head_gemm: gate bf16 like y, or [T, heads]");
  c10::cuda::CUDAGuard g(x.device());
  check(b2_head_gemm_bf16(x.data_ptr(), w.data_ptr(), y.data_ptr(), gate.has_value() ? gate->data_ptr() : nullptr, as_int(x.size(0)), as_int(heads),
                          as_int(w.size(0) / heads), as_int(w.size(1)), x.stride(0), w.stride(0), y.stride(0), gate.has_value() ? gate->stride(0) : 0,
                          by_head ? 1 : 0, status_ptr(status), cur_stream()), "head_gemm");
}

void moe_route(const at::Tensor& logits, at::Tensor& weights, at::Tensor& ids, at::Tensor& place, at::Tensor& counts, int64_t experts, int64_t scoring,
               bool norm_top, double scale, const OptTensor& correction, int64_t groups, int64_t keep, int64_t identity) {
  need(logits.is_cuda() && logits.scalar_type() == at::kFloat && rows_of(logits) && logits.size(1) >= experts + identity, "moe_route: logits f32 [T, >= experts + identity]");
  if (correction.has_value()) need(is_f32(*correction, experts + identity), "moe_route: correction f32 [experts + identity]");
  need(ids.dim() == 2 && is_i32(ids) && is_i32(place) && place.sizes() == ids.sizes() && is_f32(weights, ids.numel()) && ids.size(0) == logits.size(0) &&
           is_i32(counts) && counts.numel() >= experts + 1, "moe_route: weights f32, ids and place int32 [T, top], counts int32 [experts + 1]");
  c10::cuda::CUDAGuard g(logits.device());
  check(b2_moe_route(logits.data_ptr<float>(), logits.stride(0), correction.has_value() ? correction->data_ptr<float>() : nullptr, weights.data_ptr<float>(),
                     ids.data_ptr<int32_t>(), place.data_ptr<int32_t>(), counts.data_ptr<int32_t>(), as_int(logits.size(0)), as_int(experts), as_int(identity),
                     as_int(ids.size(1)), as_int(groups), as_int(keep), as_int(scoring), norm_top ? 1 : 0, static_cast<float>(scale), cur_stream()), "moe_route");
}

void moe_gather(const at::Tensor& x, const at::Tensor& ids, const at::Tensor& place, at::Tensor& counts, at::Tensor& slot, at::Tensor& xs, at::Tensor& tiles,
                at::Tensor& n_tiles, int64_t experts, int64_t bn, const OptTensor& status, const OptTensor& weights) {
  need(is_act(x) && x.dim() == 2 && x.is_contiguous() && xs.scalar_type() == x.scalar_type() && xs.is_cuda() && xs.is_contiguous(), "moe_gather: x [T, W], xs [T * top, W]");
  const int64_t T = x.size(0), top = ids.size(1);
  need(is_i32(ids) && is_i32(place) && is_i32(slot) && ids.numel() == T * top && place.numel() == T * top && slot.numel() == T * top &&
           xs.numel() == T * top * x.size(1), "moe_gather: ids, place, slot int32 [T, top]");
  need(bn >= 1 && is_i32(counts) && counts.numel() >= experts + 1 && is_i32(tiles) && tiles.numel() >= 4 * (experts + T * top / bn) && is_i32(n_tiles),
       "moe_gather: counts [experts + 1], tiles int32 [experts + T * top / bn, 4], n_tiles int32");
  if (weights.has_value()) need(is_f32(*weights, T * top), "moe_gather: weights f32 [T, top]");
  c10::cuda::CUDAGuard g(x.device());
  check(b2_moe_gather(x.data_ptr(), ids.data_ptr<int32_t>(), place.data_ptr<int32_t>(), weights.has_value() ? weights->data_ptr<float>() : nullptr, counts.data_ptr<int32_t>(), slot.data_ptr<int32_t>(), xs.data_ptr(),
                      tiles.data_ptr<int32_t>(), n_tiles.data_ptr<int32_t>(), as_int(T), as_int(experts), as_int(top), as_int(x.size(1)), as_int(bn),
                      x.scalar_type() == at::kFloat ? 1 : 0, status_ptr(status), cur_stream()), "moe_gather");
}

void moe_tiles_gemm(const at::Tensor& x, const at::Tensor& w, const at::Tensor& tiles, const at::Tensor& n_tiles, at::Tensor& y, int64_t epilogue, int64_t bn,
                    const c10::optional<std::array<double, 4>>& act, const OptTensor& status) {
  need(is_act(x) && x.dim() == 2 && x.is_contiguous() && w.scalar_type() == x.scalar_type() && w.dim() == 3 && w.is_contiguous() && w.size(2) == x.size(1) &&
           y.scalar_type() == x.scalar_type() && y.is_contiguous() && y.dim() == 2 && y.size(0) == x.size(0) && is_i32(tiles) && is_i32(n_tiles) && tiles.dim() == 2 &&
           tiles.size(1) == 4, "moe_tiles_gemm: x [R, K], w [experts, N, K], y [R, N]; int32 tiles [n, 4]");
  const int64_t n = w.size(1);
  need(y.size(1) == (epilogue == B2_EPI_SWIGLU ? n / 2 : n), "moe_tiles_gemm: output width");
  c10::cuda::CUDAGuard g(x.device());
  if (x.scalar_type() == at::kFloat) {
    need(epilogue != B2_EPI_SWIGLU && bn <= 64, "moe_tiles_gemm: the f32 form has no gated unit and takes tiles of at most 64 rows");
    check(b2_moe_tiles_gemm_f32(x.data_ptr<float>(), w.data_ptr<float>(), tiles.data_ptr<int32_t>(), n_tiles.data_ptr<int32_t>(), y.data_ptr<float>(),
                                as_int(tiles.size(0)), as_int(n), as_int(x.size(1)), as_int(epilogue), cur_stream()), "moe_tiles_gemm_f32");
    return;
  }
  B2EpiAct a{};
  if (act.has_value()) a = {static_cast<float>((*act)[0]), static_cast<float>((*act)[1]), static_cast<float>((*act)[2]), static_cast<float>((*act)[3])};
  check(b2_moe_tiles_gemm_bf16(x.data_ptr(), w.data_ptr(), tiles.data_ptr<int32_t>(), n_tiles.data_ptr<int32_t>(), y.data_ptr(), as_int(x.size(0)),
                               as_int(w.size(0)), as_int(n), as_int(x.size(1)), as_int(epilogue), act.has_value() ? &a : nullptr, as_int(bn),
                               status_ptr(status), cur_stream()), "moe_tiles_gemm");
}
}  // namespace

void bind_latent(py::module_& m) {
  m.def("latent_write", &latent_write, py::arg("c"), py::arg("weight"), py::arg("eps"), py::arg("slots"), py::arg("cache"), py::arg("status") = py::none(),
        py::arg("k") = py::none(), py::arg("q") = py::none(), py::arg("heads") = 0, py::arg("q_off") = 0, py::arg("column") = 0, py::arg("cos_sin") = py::none(),
        py::arg("positions") = py::none());
  m.def("latent_gather", &latent_gather);
  m.def("latent_attend", &latent_attend, py::arg("q"), py::arg("cache"), py::arg("out"), py::arg("row_ctx"), py::arg("tables"), py::arg("row_seq"),
        py::arg("workspace"), py::arg("heads"), py::arg("splits"), py::arg("scale"), py::arg("status") = py::none(), py::arg("latent") = 0, py::arg("window") = 0);
  m.def("token_rows", &token_rows);
  m.def("head_gemm", &head_gemm);
  m.def("moe_route", &moe_route, py::arg("logits"), py::arg("weights"), py::arg("ids"), py::arg("place"), py::arg("counts"), py::arg("experts"),
        py::arg("scoring"), py::arg("norm_top"), py::arg("scale"), py::arg("correction") = py::none(), py::arg("groups") = 1, py::arg("keep") = 1,
        py::arg("identity") = 0);
  m.def("moe_gather", &moe_gather, py::arg("x"), py::arg("ids"), py::arg("place"), py::arg("counts"), py::arg("slot"), py::arg("xs"), py::arg("tiles"),
        py::arg("n_tiles"), py::arg("experts"), py::arg("bn"), py::arg("status") = py::none(), py::arg("weights") = py::none());
  m.def("moe_tiles_gemm", &moe_tiles_gemm);
}
