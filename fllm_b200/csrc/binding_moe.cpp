// torch.ops.fllm_b200 bindings of the mixture-of-experts kernels.
#include <ATen/ATen.h>
#include <c10/cuda/CUDAGuard.h>
#include <c10/cuda/CUDAStream.h>
#include <torch/library.h>

#include <algorithm>

#include "fllm_ops.h"

namespace {
using at::Tensor;
using c10::optional;
inline cudaStream_t cur_stream() { return c10::cuda::getCurrentCUDAStream().stream(); }
inline const void* optp(const optional<Tensor>& t) { return t.has_value() && t->defined() ? t->data_ptr() : nullptr; }

void moe_route(const Tensor& logits, const optional<Tensor>& bias, int64_t k, bool softmax_all, Tensor ids, Tensor weights) {
  TORCH_CHECK(logits.is_cuda() && logits.scalar_type() == at::kBFloat16 && logits.dim() == 2 && logits.stride(1) == 1, "logits: bf16 rows");
  TORCH_CHECK(ids.scalar_type() == at::kInt && weights.scalar_type() == at::kFloat && ids.is_contiguous() && weights.is_contiguous(), "ids int32, weights fp32");
  c10::cuda::CUDAGuard guard(logits.device());
  fllm::moe_route(logits.data_ptr(), logits.stride(0), optp(bias), (int)logits.size(0), (int)logits.size(1), (int)k,
                  softmax_all ? 1 : 0, ids.data_ptr<int>(), weights.data_ptr<float>(), cur_stream());
}

void moe_route_scored(const Tensor& logits, const optional<Tensor>& select_bias, int64_t k, int64_t score_kind, bool renorm, double scale,
                      Tensor ids, Tensor weights) {
  TORCH_CHECK(logits.is_cuda() && logits.scalar_type() == at::kBFloat16 && logits.dim() == 2 && logits.stride(1) == 1, "logits: bf16 rows");
  TORCH_CHECK(ids.scalar_type() == at::kInt && weights.scalar_type() == at::kFloat && ids.is_contiguous() && weights.is_contiguous(), "ids int32, weights fp32");
  const float* sb = nullptr;
  if (select_bias.has_value() && select_bias->defined()) {
    TORCH_CHECK(select_bias->scalar_type() == at::kFloat && select_bias->is_contiguous() && select_bias->numel() == logits.size(1), "select_bias: fp32 [experts]");
    sb = select_bias->data_ptr<float>();
  }
  c10::cuda::CUDAGuard guard(logits.device());
  fllm::moe_route_scored(logits.data_ptr(), logits.stride(0), sb, (int)logits.size(0), (int)logits.size(1), (int)k, (int)score_kind,
                         renorm ? 1 : 0, (float)scale, ids.data_ptr<int>(), weights.data_ptr<float>(), cur_stream());
}

// logits fp32 [T, ld], or their split-K partial sums [splits][T][ld] in `workspace`; gate_out (optional) [T]: the sigmoid of column `experts`
void moe_route_fp32(const optional<Tensor>& logits, const optional<Tensor>& workspace, int64_t splits, int64_t ld, int64_t experts, int64_t k,
                    int64_t score_kind, bool renorm, double scale, Tensor ids, Tensor weights, const optional<Tensor>& select_bias, int64_t groups,
                    int64_t keep, double masked, const optional<Tensor>& gate_out) {
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kInt && ids.dim() == 2 && ids.size(1) == k && weights.scalar_type() == at::kFloat &&
                  ids.is_contiguous() && weights.is_contiguous() && weights.numel() == ids.numel() && experts <= ld, "ids int32, weights fp32 [T, k]");
  const int64_t T = ids.size(0);
  const float* z = nullptr;
  if (splits > 0) {
    TORCH_CHECK(workspace.has_value() && workspace->is_contiguous() && workspace->nbytes() >= fllm::kLinearPartialsOffset + (size_t)splits * T * ld * 4,
                "workspace too small for the split-K partials");
    z = reinterpret_cast<const float*>(reinterpret_cast<const uint8_t*>(workspace->data_ptr()) + fllm::kLinearPartialsOffset);
  } else {
    TORCH_CHECK(logits.has_value() && logits->is_cuda() && logits->scalar_type() == at::kFloat && logits->is_contiguous() && logits->dim() == 2 &&
                    logits->size(0) == T && logits->size(1) == ld, "logits: contiguous fp32 [T, ld]");
    z = logits->data_ptr<float>();
  }
  const float* sb = nullptr;
  if (select_bias.has_value() && select_bias->defined()) {
    TORCH_CHECK(select_bias->is_cuda() && select_bias->scalar_type() == at::kFloat && select_bias->is_contiguous() && select_bias->numel() == experts, "select_bias: fp32 [experts]");
    sb = select_bias->data_ptr<float>();
  }
  float* gate = nullptr;
  if (gate_out.has_value() && gate_out->defined()) {
    TORCH_CHECK(gate_out->is_cuda() && gate_out->scalar_type() == at::kFloat && gate_out->is_contiguous() && gate_out->numel() == T && experts < ld, "gate_out: fp32 [T]");
    gate = gate_out->data_ptr<float>();
  }
  c10::cuda::CUDAGuard guard(ids.device());
  fllm::moe_route_fp32(z, (int)std::max<int64_t>(splits, 1), T * ld, ld, (int)T, (int)experts, (int)k, (int)score_kind, renorm ? 1 : 0, (float)scale,
                       ids.data_ptr<int>(), weights.data_ptr<float>(), cur_stream(), sb, fllm::RouteGroups{(int)groups, (int)keep, (float)masked}, gate);
}

void moe_align(const Tensor& ids, int64_t experts, int64_t expert_lo, int64_t expert_hi, int64_t bn, Tensor row_of,
               Tensor token_of, Tensor tile_expert, Tensor tile_row0, Tensor num_tiles, const optional<Tensor>& weights,
               const optional<Tensor>& row_weight) {
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kInt && ids.dim() == 2 && ids.is_contiguous(), "ids: [tokens, k] int32");
  TORCH_CHECK(num_tiles.numel() >= 2 && expert_lo >= 0 && expert_lo <= expert_hi && expert_hi <= experts, "num_tiles needs two ints; a range of the experts");
  const bool weighed = row_weight.has_value() && row_weight->defined();
  TORCH_CHECK(!weighed || (weights.has_value() && weights->scalar_type() == at::kFloat && weights->is_contiguous() && weights->numel() == ids.numel() &&
                           row_weight->scalar_type() == at::kFloat && row_weight->is_contiguous() && row_weight->numel() >= token_of.numel()),
              "weights fp32 like ids, row_weight fp32 like token_of");
  c10::cuda::CUDAGuard guard(ids.device());
  fllm::moe_align(ids.data_ptr<int>(), (int)ids.size(0), (int)ids.size(1), (int)expert_lo, (int)expert_hi,
                  (int)bn, row_of.data_ptr<int>(), token_of.data_ptr<int>(), (int)token_of.numel(),
                  tile_expert.data_ptr<int>(), tile_row0.data_ptr<int>(), num_tiles.data_ptr<int>(),
                  (int)tile_expert.numel(), cur_stream(), weighed ? weights->data_ptr<float>() : nullptr,
                  weighed ? row_weight->data_ptr<float>() : nullptr);
}

inline bool f32_rows(const Tensor& t) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat) && t.dim() == 2 && t.stride(1) == 1, "rows of bf16 or fp32");
  return t.scalar_type() == at::kFloat;
}

void moe_gather(const Tensor& x, const Tensor& token_of, Tensor xp, const optional<Tensor>& row_weight) {
  const bool f32 = f32_rows(x);
  TORCH_CHECK(xp.scalar_type() == x.scalar_type() && xp.is_contiguous() && xp.size(1) == x.size(1) && x.size(1) % 8 == 0 && x.stride(0) % 8 == 0 &&
                  token_of.numel() >= xp.size(0), "moe_gather: shapes");
  const float* rw = nullptr;
  if (row_weight.has_value() && row_weight->defined()) {
    TORCH_CHECK(row_weight->scalar_type() == at::kFloat && row_weight->is_contiguous() && row_weight->numel() >= xp.size(0), "row_weight: fp32 per row");
    rw = row_weight->data_ptr<float>();
  }
  c10::cuda::CUDAGuard guard(x.device());
  fllm::moe_gather(x.data_ptr(), x.stride(0), token_of.data_ptr<int>(), xp.data_ptr(), (int)xp.size(0), (int)x.size(1), cur_stream(), rw, f32 ? 1 : 0);
}

// fp32: w_stack [experts, n_out, K], xp [rows_cap, K], y [rows_cap, n_out], tiles of 64 rows
void moe_grouped_linear_f32(const Tensor& xp, const Tensor& w_stack, Tensor y, const Tensor& tile_expert, const Tensor& tile_row0, const Tensor& num_tiles,
                            int64_t bn) {
  TORCH_CHECK(bn == 64 && f32_rows(xp) && f32_rows(y) && w_stack.scalar_type() == at::kFloat && w_stack.dim() == 3 && w_stack.is_contiguous() &&
                  xp.size(1) == w_stack.size(2) && y.size(0) == xp.size(0) && y.size(1) == w_stack.size(1), "w_stack [E, n, k], xp [rows, k], y [rows, n]: fp32");
  fllm::GemmF32Params p{};
  p.a = xp.data_ptr<float>(), p.a_t = xp.stride(0), p.a_k = 1;
  p.b = w_stack.data_ptr<float>(), p.b_b = w_stack.stride(0), p.b_n = w_stack.stride(1), p.b_k = 1;
  p.c = y.data_ptr<float>(), p.c_t = y.stride(0);
  p.batch = 1, p.T = (int)xp.size(0), p.N = (int)w_stack.size(1), p.K = (int)xp.size(1);
  c10::cuda::CUDAGuard guard(xp.device());
  fllm::moe_grouped_f32(p, tile_expert.data_ptr<int>(), tile_row0.data_ptr<int>(), num_tiles.data_ptr<int>(), (int)tile_expert.numel(), cur_stream());
}

// w_stack: [experts, n_out, K]; xp: [rows_cap, K]; y: [rows_cap, n_out]
int64_t moe_grouped_linear(const Tensor& xp, const Tensor& w_stack, const optional<Tensor>& bias_stack, Tensor y,
                           const Tensor& tile_expert, const Tensor& tile_row0, const Tensor& num_tiles, int64_t bn,
                           const optional<Tensor>& status) {
  TORCH_CHECK(w_stack.dim() == 3 && w_stack.is_contiguous() && w_stack.scalar_type() == at::kBFloat16, "w_stack: contiguous [E, n, k] bf16");
  TORCH_CHECK(xp.dim() == 2 && xp.stride(1) == 1 && xp.size(1) == w_stack.size(2), "xp: [rows, k]");
  TORCH_CHECK(y.dim() == 2 && y.stride(1) == 1 && y.size(0) == xp.size(0) && y.size(1) == w_stack.size(1), "y: [rows, n]");
  c10::cuda::CUDAGuard guard(xp.device());
  int* st = status.has_value() && status->defined() ? status->data_ptr<int>() : nullptr;
  return fllm::moe_grouped_linear_bf16(xp.data_ptr(), xp.stride(0), w_stack.data_ptr(), w_stack.stride(1), optp(bias_stack),
                                       y.data_ptr(), y.stride(0), (int)xp.size(0), (int)w_stack.size(1), (int)w_stack.size(2),
                                       (int)w_stack.size(0), tile_expert.data_ptr<int>(), tile_row0.data_ptr<int>(),
                                       num_tiles.data_ptr<int>(), (int)tile_expert.numel(), (int)bn, st, cur_stream());
}

void moe_combine(const Tensor& y, const Tensor& row_of, const optional<Tensor>& weights, Tensor out, const optional<Tensor>& add,
                 const optional<Tensor>& add_gate) {
  const bool f32 = f32_rows(y), plus = add.has_value() && add->defined();
  TORCH_CHECK(out.scalar_type() == y.scalar_type() && out.stride(1) == 1 && y.size(1) == out.size(1) && y.size(1) % 4 == 0 && y.stride(0) % 4 == 0 &&
                  out.stride(0) % 4 == 0, "moe_combine: shapes");
  TORCH_CHECK(!plus || (f32_rows(*add) == f32 && add->sizes() == out.sizes() && add->stride(0) % 4 == 0), "add: rows like out");
  const bool gated = add_gate.has_value() && add_gate->defined();
  TORCH_CHECK(!gated || (plus && add_gate->is_cuda() && add_gate->scalar_type() == at::kFloat && add_gate->is_contiguous() && add_gate->numel() == out.size(0)),
              "add_gate: fp32, one per row");
  c10::cuda::CUDAGuard guard(y.device());
  fllm::moe_combine(y.data_ptr(), y.stride(0), row_of.data_ptr<int>(), weights.has_value() && weights->defined() ? weights->data_ptr<float>() : nullptr,
                    (int)out.size(0), (int)row_of.size(1), out.data_ptr(), out.stride(0), (int)out.size(1), cur_stream(), plus ? add->data_ptr() : nullptr,
                    plus ? add->stride(0) : 0, f32 ? 1 : 0, gated ? add_gate->data_ptr<float>() : nullptr);
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("moe_route_scored(Tensor logits, Tensor? select_bias, int k, int score_kind, bool renorm, float scale, Tensor(a!) ids, Tensor(b!) weights) -> ()",
        &moe_route_scored);
  m.def("moe_route(Tensor logits, Tensor? bias, int k, bool softmax_all, Tensor(a!) ids, Tensor(b!) weights) -> ()", &moe_route);
  m.def("moe_route_fp32(Tensor? logits, Tensor? workspace, int splits, int ld, int experts, int k, int score_kind, bool renorm, float scale, "
        "Tensor(a!) ids, Tensor(b!) weights, Tensor? select_bias=None, int groups=1, int keep=1, float masked=0.0, Tensor(c!)? gate_out=None) -> ()",
        &moe_route_fp32);
  m.def("moe_grouped_linear_f32(Tensor xp, Tensor w_stack, Tensor(a!) y, Tensor tile_expert, Tensor tile_row0, Tensor num_tiles, int bn) -> ()",
        &moe_grouped_linear_f32);
  m.def("moe_align(Tensor ids, int experts, int expert_lo, int expert_hi, int bn, Tensor(a!) row_of, Tensor(b!) token_of, Tensor(c!) tile_expert, Tensor(d!) tile_row0, Tensor(e!) num_tiles, Tensor? weights=None, Tensor(f!)? row_weight=None) -> ()", &moe_align);
  m.def("moe_gather(Tensor x, Tensor token_of, Tensor(a!) xp, Tensor? row_weight=None) -> ()", &moe_gather);
  m.def("moe_grouped_linear(Tensor xp, Tensor w_stack, Tensor? bias_stack, Tensor(a!) y, Tensor tile_expert, Tensor tile_row0, Tensor num_tiles, int bn, Tensor? status) -> int", &moe_grouped_linear);
  m.def("moe_combine(Tensor y, Tensor row_of, Tensor? weights, Tensor(a!) out, Tensor? add=None, Tensor? add_gate=None) -> ()", &moe_combine);
}
