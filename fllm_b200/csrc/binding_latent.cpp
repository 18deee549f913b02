// torch.ops.fllm_b200 bindings of the hyper-connected residual streams (streams.cu) and latent attention of any size
// (attention_latent.cu).
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
inline at::ScalarType act_type(const Tensor& t) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat), "activations are bf16 or fp32 on a GPU");
  return t.scalar_type();
}
inline const float* coef(const optional<Tensor>& t, int64_t n) {
  if (!given(t)) return nullptr;
  TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kFloat && t->is_contiguous() && t->numel() == n, "stream coefficients: contiguous fp32");
  return t->data_ptr<float>();
}

// x fp32 [rows, S, ld]. Start: ids + table. Otherwise y [rows, ld] or, with splits > 0, its split-K partial sums in `workspace`.
// h [outputs, ld]; rows (int32) selects the rows that are read; `write` stores the updated streams.
void stream_mix_norm(Tensor x, const optional<Tensor>& ids, const optional<Tensor>& table, const optional<Tensor>& y,
                     const optional<Tensor>& workspace, int64_t splits, const optional<Tensor>& mix, const optional<Tensor>& out,
                     const Tensor& in, const optional<Tensor>& rows, const Tensor& norm_w, const optional<Tensor>& norm_b, Tensor h,
                     int64_t width, double eps, bool rms, bool write) {
  const auto ty = act_type(h);
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == at::kFloat && x.dim() == 3 && x.is_contiguous(), "x: contiguous fp32 [rows, streams, ld]");
  const int64_t n = x.size(0), S = x.size(1), ld = x.size(2);
  TORCH_CHECK(h.dim() == 2 && h.stride(1) == 1 && h.size(1) == ld && norm_w.scalar_type() == ty && norm_w.is_contiguous() && norm_w.numel() == ld,
              "h rows and norm weights have the padded width of the streams");
  TORCH_CHECK(!given(norm_b) || (norm_b->scalar_type() == ty && norm_b->is_contiguous() && norm_b->numel() == ld), "norm bias");
  fllm::StreamMixParams p{};
  p.x = x.data_ptr<float>();
  p.in = coef(in, S);
  if (given(ids)) {
    TORCH_CHECK(i32(*ids) && ids->numel() == n && given(table) && table->scalar_type() == ty && table->dim() == 2 && table->stride(1) == 1 &&
                    table->size(1) == ld, "ids int32 [rows], table [vocab, ld]");
    p.ids = ids->data_ptr<int>();
    p.table = table->data_ptr();
    p.vocab = (int)table->size(0);
    p.ld_table = table->stride(0);
  } else {
    TORCH_CHECK(given(mix) && given(out), "an update needs mix and out");
    p.mix = coef(mix, S * S);
    p.out = coef(out, S);
    if (splits > 0) {
      TORCH_CHECK(given(workspace) && workspace->is_contiguous() &&
                      workspace->nbytes() >= fllm::kLinearPartialsOffset + (size_t)splits * n * ld * 4, "workspace too small for the split-K partials");
      p.partials = reinterpret_cast<const float*>(reinterpret_cast<const uint8_t*>(workspace->data_ptr()) + fllm::kLinearPartialsOffset);
      p.splits = (int)splits;
      p.plane = n * ld;
    } else {
      TORCH_CHECK(given(y) && y->scalar_type() == ty && y->dim() == 2 && y->stride(1) == 1 && y->size(0) == n && y->size(1) == ld, "y: [rows, ld] like h");
      p.y = y->data_ptr();
      p.ld_y = y->stride(0);
    }
  }
  p.n_out = (int)n;
  if (given(rows)) {
    TORCH_CHECK(i32(*rows) && !write, "rows: int32; a selection of rows does not update the streams");
    p.rows = rows->data_ptr<int>();
    p.n_out = (int)rows->numel();
  }
  TORCH_CHECK(h.size(0) == p.n_out, "h: one row per output");
  p.norm_w = norm_w.data_ptr();
  p.norm_b = given(norm_b) ? norm_b->data_ptr() : nullptr;
  p.h = h.data_ptr();
  p.ld_h = h.stride(0);
  p.streams = (int)S, p.width = (int)width, p.ld = (int)ld;
  p.eps = (float)eps;
  p.rms = rms ? 1 : 0, p.write = write ? 1 : 0, p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(h.device());
  fllm::stream_mix_norm(p, cur_stream());
}

// q rows [T, >= H * head], ckv rows [T, >= R + dr] (none: another layer's rows are used), cache [blocks, block_size, W],
// q_out [H, T, W]
void latent_prepare(const optional<Tensor>& ckv, const Tensor& q, int64_t head, int64_t rope_offset, const Tensor& positions,
                    const Tensor& slots, const Tensor& inv_freq, double attn_factor, const optional<Tensor>& norm_w, double eps, Tensor cache,
                    Tensor q_out, int64_t R, int64_t style) {
  const auto ty = act_type(q);
  const int64_t T = q.size(0), H = q_out.size(0), W = q_out.size(2), dr = 2 * inv_freq.numel();
  TORCH_CHECK(q.dim() == 2 && q.stride(1) == 1 && q.size(1) >= H * head && rope_offset + dr <= head, "q: rows of H heads");
  TORCH_CHECK(q_out.dim() == 3 && q_out.is_contiguous() && q_out.scalar_type() == ty && q_out.size(1) == T, "q_out: contiguous [H, T, W]");
  TORCH_CHECK(cache.dim() == 3 && cache.is_contiguous() && cache.scalar_type() == ty && cache.size(2) == W && R + dr <= W, "cache: [blocks, block_size, W]");
  TORCH_CHECK(i32(positions) && i32(slots) && positions.numel() >= T && slots.numel() >= T && inv_freq.scalar_type() == at::kFloat && inv_freq.is_contiguous(),
              "positions, slots int32 [T]; inv_freq fp32");
  fllm::LatentPrepareParams p{};
  if (given(ckv)) {
    TORCH_CHECK(ckv->scalar_type() == ty && ckv->dim() == 2 && ckv->stride(1) == 1 && ckv->size(0) == T && ckv->size(1) >= R + dr && given(norm_w) &&
                    norm_w->scalar_type() == ty && norm_w->is_contiguous() && norm_w->numel() == R, "ckv: [T, >= R + dr], norm_w [R]");
    p.ckv = ckv->data_ptr();
    p.ld_ckv = ckv->stride(0);
    p.norm_w = norm_w->data_ptr();
  }
  p.q = q.data_ptr(), p.ld_q = q.stride(0), p.q_head = (int)head, p.q_rope_offset = (int)rope_offset;
  p.positions = positions.data_ptr<int>(), p.slots = slots.data_ptr<int>(), p.inv_freq = inv_freq.data_ptr<float>();
  p.attn_factor = (float)attn_factor, p.eps = (float)eps;
  p.cache = cache.data_ptr(), p.q_out = q_out.data_ptr(), p.q_out_h = q_out.stride(0);
  p.tokens = (int)T, p.H = (int)H, p.R = (int)R, p.dr = (int)dr, p.W = (int)W, p.style = (int)style, p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(q.device());
  fllm::latent_prepare(p, cur_stream());
}

int64_t attention_latent_splits(int64_t num_seqs, int64_t tokens, int64_t max_q_len, int64_t H, int64_t max_kv_len) {
  return fllm::attention_latent_splits((int)num_seqs, (int)tokens, (int)max_q_len, (int)H, (int)max_kv_len);
}
int64_t attention_latent_workspace_bytes(int64_t tokens, int64_t H, int64_t R, int64_t splits) {
  return (int64_t)fllm::attention_latent_workspace_bytes((int)tokens, (int)H, (int)R, (int)splits);
}

// q [H, T, W] contiguous, out [H, T, R] (unit inner stride); returns the number of kernels launched
int64_t attention_latent(const Tensor& q, const Tensor& cache, const Tensor& block_tables, const Tensor& row_seq, const Tensor& positions,
                         const Tensor& q_starts, Tensor out, int64_t num_seqs, int64_t max_q_len, double scale, int64_t splits,
                         const optional<Tensor>& workspace, bool tensor_cores) {
  const auto ty = act_type(q);
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && cache.dim() == 3 && cache.is_contiguous() && cache.scalar_type() == ty && cache.size(2) == q.size(2),
              "q [H, T, W], cache [blocks, block_size, W]: contiguous");
  const int64_t H = q.size(0), T = q.size(1);
  TORCH_CHECK(out.dim() == 3 && out.stride(2) == 1 && out.scalar_type() == ty && out.size(0) == H && out.size(1) == T && out.size(2) <= q.size(2), "out: [H, T, R]");
  TORCH_CHECK(block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 && block_tables.stride(1) == 1 && i32(row_seq) && i32(positions) &&
                  i32(q_starts) && row_seq.numel() >= T && positions.numel() >= T && q_starts.numel() >= num_seqs + 1,
              "block_tables [B, max_blocks], row_seq [T], positions [T], q_starts [B + 1]: int32");
  void* ws = nullptr;
  size_t ws_bytes = 0;
  if (given(workspace)) {
    TORCH_CHECK(workspace->is_cuda() && workspace->is_contiguous(), "workspace: contiguous CUDA tensor");
    ws = workspace->data_ptr();
    ws_bytes = workspace->nbytes();
  }
  fllm::LatentAttnParams p{};
  p.q = q.data_ptr(), p.q_h = q.stride(0), p.cache = cache.data_ptr();
  p.block_tables = block_tables.data_ptr<int>(), p.max_blocks = (int)block_tables.stride(0);
  p.row_seq = row_seq.data_ptr<int>(), p.positions = positions.data_ptr<int>(), p.q_starts = q_starts.data_ptr<int>();
  p.out = out.data_ptr(), p.o_h = out.stride(0), p.o_t = out.stride(1);
  p.tokens = (int)T, p.num_seqs = (int)num_seqs, p.max_q_len = (int)max_q_len, p.H = (int)H, p.R = (int)out.size(2), p.W = (int)q.size(2);
  p.block_size = (int)cache.size(1), p.scale = (float)scale, p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(q.device());
  return fllm::attention_latent(p, (int)splits, ws, ws_bytes, tensor_cores, cur_stream());
}

// o [H, T, dv], gate [T, H] rows or none, out [T, >= H * dv]
void head_gate(const Tensor& o, const optional<Tensor>& gate, Tensor out) {
  const auto ty = act_type(o);
  TORCH_CHECK(o.dim() == 3 && o.stride(2) == 1 && out.scalar_type() == ty && out.dim() == 2 && out.stride(1) == 1 && out.size(0) == o.size(1) &&
                  out.size(1) >= o.size(0) * o.size(2), "o [H, T, dv], out [T, >= H * dv]");
  const void* g = nullptr;
  long long ldg = 0;
  if (given(gate)) {
    TORCH_CHECK(gate->scalar_type() == ty && gate->dim() == 2 && gate->stride(1) == 1 && gate->size(0) == o.size(1) && gate->size(1) >= o.size(0), "gate: [T, H]");
    g = gate->data_ptr();
    ldg = gate->stride(0);
  }
  c10::cuda::CUDAGuard guard(o.device());
  fllm::head_gate(o.data_ptr(), o.stride(0), o.stride(1), g, ldg, out.data_ptr(), out.stride(0), (int)o.size(1), (int)o.size(0), (int)o.size(2),
                  (int)out.size(1), ty == at::kFloat ? 1 : 0, cur_stream());
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("stream_mix_norm(Tensor(a!) x, Tensor? ids, Tensor? table, Tensor? y, Tensor? workspace, int splits, Tensor? mix, Tensor? out, Tensor in_, "
        "Tensor? rows, Tensor norm_w, Tensor? norm_b, Tensor(b!) h, int width, float eps, bool rms, bool write) -> ()", &stream_mix_norm);
  m.def("latent_prepare(Tensor? ckv, Tensor q, int head, int rope_offset, Tensor positions, Tensor slots, Tensor inv_freq, float attn_factor, "
        "Tensor? norm_w, float eps, Tensor(a!) cache, Tensor(b!) q_out, int R, int style) -> ()", &latent_prepare);
  m.def("attention_latent_splits(int num_seqs, int tokens, int max_q_len, int H, int max_kv_len) -> int", &attention_latent_splits);
  m.def("attention_latent_workspace_bytes(int tokens, int H, int R, int splits) -> int", &attention_latent_workspace_bytes);
  m.def("attention_latent(Tensor q, Tensor cache, Tensor block_tables, Tensor row_seq, Tensor positions, Tensor q_starts, Tensor(a!) out, int num_seqs, "
        "int max_q_len, float scale, int splits, Tensor? workspace, bool tensor_cores) -> int", &attention_latent);
  m.def("head_gate(Tensor o, Tensor? gate, Tensor(a!) out) -> ()", &head_gate);
}
