// torch.ops.fllm_b200 bindings of the fp32 residual with norms behind the sum or on what is added (postnorm.cu).
#include <ATen/ATen.h>
#include <c10/cuda/CUDAGuard.h>
#include <c10/cuda/CUDAStream.h>
#include <torch/library.h>

#include "fllm_ops.h"

namespace {
using at::Tensor;
using c10::optional;
inline cudaStream_t cur_stream() { return c10::cuda::getCurrentCUDAStream().stream(); }
inline bool given(const optional<Tensor>& t) { return t.has_value() && t->defined(); }
inline bool i32(const Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous(); }
inline bool rows_of(const Tensor& t, at::ScalarType ty) { return t.is_cuda() && t.scalar_type() == ty && t.dim() == 2 && t.stride(1) == 1; }
inline bool f32(const Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous(); }
inline at::ScalarType act_type(const Tensor& t) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat), "activations are bf16 or fp32 on a GPU");
  return t.scalar_type();
}
// split-K partial sums [splits][rows][cols] a projection left in the workspace
inline const float* partial_sums(const optional<Tensor>& workspace, int64_t splits, int64_t rows, int64_t cols) {
  TORCH_CHECK(given(workspace) && workspace->is_contiguous() && workspace->nbytes() >= fllm::kLinearPartialsOffset + (size_t)splits * rows * cols * 4,
              "workspace too small for the split-K partials");
  return reinterpret_cast<const float*>(reinterpret_cast<const uint8_t*>(workspace->data_ptr()) + fllm::kLinearPartialsOffset);
}

// x fp32 [rows, ld]. Start: ids + table. Otherwise y [rows, ld] or, with splits > 0, its split-K partial sums in `workspace`;
// with pair_a half the sum of pair_a and y, each over its root mean square times its weight.
void postnorm(Tensor x, const optional<Tensor>& ids, const optional<Tensor>& table, double scale, const optional<Tensor>& y,
              const optional<Tensor>& workspace, int64_t splits, bool add, double alpha, const optional<Tensor>& norm_w, const optional<Tensor>& final_w,
              double final_scale, const optional<Tensor>& rows, Tensor h, int64_t width, double eps, bool write, const optional<Tensor>& pair_a,
              const optional<Tensor>& pair_wa, const optional<Tensor>& pair_wb) {
  const auto ty = act_type(h);
  TORCH_CHECK(f32(x) && x.dim() == 2, "x: contiguous fp32 [rows, ld]");
  const int64_t n = x.size(0), ld = x.size(1);
  TORCH_CHECK(rows_of(h, ty) && h.size(1) == ld, "h: rows of the residual's padded width");
  auto vec = [&](const optional<Tensor>& t) -> const void* {
    TORCH_CHECK(t->scalar_type() == ty && t->is_cuda() && t->is_contiguous() && t->numel() == ld, "norm weights: the padded width, like h");
    return t->data_ptr();
  };
  fllm::PostNormParams p{};
  p.x = x.data_ptr<float>();
  if (given(ids)) {
    TORCH_CHECK(i32(*ids) && ids->numel() == n && given(table) && rows_of(*table, ty) && table->size(1) == ld, "ids int32 [rows], table [vocab, ld]");
    p.ids = ids->data_ptr<int>(), p.table = table->data_ptr(), p.vocab = (int)table->size(0), p.ld_table = table->stride(0), p.scale = (float)scale;
  } else {
    TORCH_CHECK(given(norm_w), "an update needs a norm weight");
    p.norm_w = vec(norm_w);
    if (splits > 0) {
      p.partials = partial_sums(workspace, splits, n, ld);
      p.splits = (int)splits, p.plane = n * ld;
    } else {
      TORCH_CHECK(given(y) && rows_of(*y, ty) && y->size(0) == n && y->size(1) == ld, "y: [rows, ld] like h");
      p.y = y->data_ptr(), p.ld_y = y->stride(0);
    }
    if (given(pair_a)) {
      TORCH_CHECK(rows_of(*pair_a, ty) && pair_a->size(0) == n && pair_a->size(1) == ld && given(pair_wa) && given(pair_wb), "pair_a: [rows, ld] like h, with two weights");
      p.pair_a = pair_a->data_ptr(), p.ld_pair = pair_a->stride(0), p.pair_wa = vec(pair_wa), p.pair_wb = vec(pair_wb);
    }
  }
  p.n_out = (int)n;
  if (given(rows)) {
    TORCH_CHECK(i32(*rows) && !write, "rows: int32; a selection of rows does not update the residual");
    p.rows = rows->data_ptr<int>(), p.n_out = (int)rows->numel();
  }
  TORCH_CHECK(h.size(0) == p.n_out, "h: one row per output");
  if (given(final_w)) p.final_w = vec(final_w);
  p.add = add ? 1 : 0, p.alpha = (float)alpha, p.final_scale = (float)final_scale;
  p.h = h.data_ptr(), p.ld_h = h.stride(0), p.width = (int)width, p.ld = (int)ld, p.eps = (float)eps;
  p.write = write ? 1 : 0, p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(h.device());
  fllm::postnorm(p, cur_stream());
}

// out [T, cols] = gelu_tanh(gate) * table[ids, offset : offset + dim], zeros behind; gate [T, cols] or its split-K partial sums
void side_gate(const optional<Tensor>& gate, const optional<Tensor>& workspace, int64_t splits, const Tensor& ids, const Tensor& table, int64_t offset,
               int64_t dim, Tensor out) {
  const auto ty = act_type(out);
  TORCH_CHECK(rows_of(out, ty) && rows_of(table, ty) && i32(ids) && ids.numel() >= out.size(0) && offset >= 0 && dim <= out.size(1) &&
                  offset + dim <= table.size(1), "out [T, cols >= dim], table [vocab, >= offset + dim], ids int32 [T]");
  fllm::SideGateParams p{};
  const int64_t T = out.size(0), cols = out.size(1);
  if (splits > 0) {
    p.partials = partial_sums(workspace, splits, T, cols);
    p.splits = (int)splits, p.plane = T * cols;
  } else {
    TORCH_CHECK(given(gate) && rows_of(*gate, ty) && gate->size(0) == T && gate->size(1) == cols, "gate: [T, cols]");
    p.gate = gate->data_ptr(), p.ld_gate = gate->stride(0);
  }
  p.ids = ids.data_ptr<int>(), p.table = table.data_ptr(), p.vocab = (int)table.size(0), p.ld_table = table.stride(0);
  p.offset = (int)offset, p.dim = (int)dim, p.cols = (int)cols, p.tokens = (int)T;
  p.out = out.data_ptr(), p.ld_out = out.stride(0), p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(out.device());
  fllm::side_gate(p, cur_stream());
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("postnorm(Tensor(a!) x, Tensor? ids, Tensor? table, float scale, Tensor? y, Tensor? workspace, int splits, bool add, float alpha, Tensor? norm_w, "
        "Tensor? final_w, float final_scale, Tensor? rows, Tensor(b!) h, int width, float eps, bool write, Tensor? pair_a=None, Tensor? pair_wa=None, Tensor? pair_wb=None) -> ()", &postnorm);
  m.def("side_gate(Tensor? gate, Tensor? workspace, int splits, Tensor ids, Tensor table, int offset, int dim, Tensor(a!) out) -> ()", &side_gate);
}
