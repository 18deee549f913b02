// torch.ops.fllm_b200 bindings of the fp32 residual with the norm in front of a sublayer (prenorm.cu).
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

// x, x_out fp32 [rows, ld] (x may be left out: the sum starts at zero); y [rows, ld] or, with splits > 0, its split-K partial sums in
// `workspace`; ids + table: rows of the table are added. With `shift` a token shift over the sequences of the step follows the norm.
void prenorm(const optional<Tensor>& x, const optional<Tensor>& x_out, const optional<Tensor>& ids, const optional<Tensor>& table,
             const optional<Tensor>& y, const optional<Tensor>& workspace, int64_t splits, const Tensor& norm_w, double w_offset, int64_t n, int64_t width,
             double eps, const optional<Tensor>& rows, Tensor h, const optional<Tensor>& shift, const optional<Tensor>& state,
             const optional<Tensor>& q_starts, const optional<Tensor>& seq_state, const optional<Tensor>& row_seq, const optional<Tensor>& positions,
             bool single) {
  TORCH_CHECK(h.is_cuda() && (h.scalar_type() == at::kBFloat16 || h.scalar_type() == at::kFloat), "activations are bf16 or fp32 on a GPU");
  const auto ty = h.scalar_type();
  TORCH_CHECK(rows_of(h, ty), "h: rows of the residual's padded width");
  const int64_t ld = h.size(1);
  auto vec = [&](const Tensor& t) -> const void* {
    TORCH_CHECK(t.scalar_type() == ty && t.is_cuda() && t.is_contiguous() && t.numel() == ld, "weights: the padded width, like h");
    return t.data_ptr();
  };
  auto res = [&](const Tensor& t) -> float* {
    TORCH_CHECK(f32(t) && t.dim() == 2 && t.size(0) == n && t.size(1) == ld, "x, x_out: contiguous fp32 [rows, ld]");
    return t.data_ptr<float>();
  };
  fllm::PreNormParams p{};
  if (given(x)) p.x = res(*x);
  if (given(x_out)) p.x_out = res(*x_out);
  if (given(ids)) {
    TORCH_CHECK(i32(*ids) && ids->numel() == n && given(table) && rows_of(*table, ty) && table->size(1) == ld, "ids int32 [rows], table [vocab, ld]");
    p.ids = ids->data_ptr<int>(), p.table = table->data_ptr(), p.vocab = (int)table->size(0), p.ld_table = table->stride(0);
  }
  if (splits > 0) {
    TORCH_CHECK(given(workspace) && workspace->is_contiguous() && workspace->nbytes() >= fllm::kLinearPartialsOffset + (size_t)splits * n * ld * 4,
                "workspace too small for the split-K partials");
    p.partials = reinterpret_cast<const float*>(reinterpret_cast<const uint8_t*>(workspace->data_ptr()) + fllm::kLinearPartialsOffset);
    p.splits = (int)splits, p.plane = n * ld;
  } else if (given(y)) {
    TORCH_CHECK(rows_of(*y, ty) && y->size(0) == n && y->size(1) == ld, "y: [rows, ld] like h");
    p.y = y->data_ptr(), p.ld_y = y->stride(0);
  }
  p.n_out = (int)n;
  if (given(rows)) {
    TORCH_CHECK(i32(*rows) && !p.x_out, "rows: int32; a selection of rows does not update the residual");
    p.rows = rows->data_ptr<int>(), p.n_out = (int)rows->numel();
  }
  TORCH_CHECK(h.size(0) == p.n_out, "h: one row per output");
  if (given(shift)) {
    TORCH_CHECK(given(state) && f32(*state) && state->dim() == 2 && state->size(1) == ld && given(q_starts) && i32(*q_starts) && given(seq_state) &&
                    i32(*seq_state) && given(row_seq) && i32(*row_seq) && given(positions) && i32(*positions) && row_seq->numel() >= n &&
                    positions->numel() >= n && q_starts->numel() == seq_state->numel() + 1 && (!single || seq_state->numel() >= n),
                "a token shift needs state rows [slots, ld] fp32 and the step's sequences");
    p.shift = vec(*shift), p.state = state->data_ptr<float>(), p.q_starts = q_starts->data_ptr<int>(), p.seq_state = seq_state->data_ptr<int>();
    p.row_seq = row_seq->data_ptr<int>(), p.positions = positions->data_ptr<int>(), p.single = single ? 1 : 0;
  }
  p.norm_w = vec(norm_w), p.w_offset = (float)w_offset, p.h = h.data_ptr(), p.ld_h = h.stride(0);
  p.width = (int)width, p.ld = (int)ld, p.eps = (float)eps, p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(h.device());
  fllm::prenorm(p, cur_stream());
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("prenorm(Tensor? x, Tensor(a!)? x_out, Tensor? ids, Tensor? table, Tensor? y, Tensor? workspace, int splits, Tensor norm_w, float w_offset, int n, "
        "int width, float eps, Tensor? rows, Tensor(b!) h, Tensor? shift, Tensor(c!)? state, Tensor? q_starts, Tensor? seq_state, Tensor? row_seq, "
        "Tensor? positions, bool single) -> ()", &prenorm);
}
