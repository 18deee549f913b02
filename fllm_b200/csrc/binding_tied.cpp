// torch.ops.fllm_b200 bindings of attention whose values are the keys (attention_tied.cu).
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

// x [T, >= k_offset + G * dim] (or its split-K partial sums, [T, q_out's type] then receives the queries), q_factor fp32 [T, H],
// cache [blocks, G, block_size, W], key_factor fp32 [blocks, G, block_size]
void tied_prepare(const optional<Tensor>& x, const optional<Tensor>& workspace, int64_t splits, int64_t width, const optional<Tensor>& q_out,
                  int64_t k_offset, int64_t dim, const Tensor& positions, const Tensor& slots, double eps, double scale, double temp_coef,
                  double temp_every, Tensor q_factor, Tensor cache, Tensor key_factor) {
  const auto ty = act_type(cache);
  TORCH_CHECK(cache.dim() == 4 && cache.is_contiguous() && f32(key_factor) && key_factor.dim() == 3 && key_factor.size(0) == cache.size(0) &&
                  key_factor.size(1) == cache.size(1) && key_factor.size(2) == cache.size(2) && cache.size(3) >= dim,
              "cache [blocks, heads, block_size, width], key_factor fp32 [blocks, heads, block_size]");
  TORCH_CHECK(f32(q_factor) && q_factor.dim() == 2, "q_factor: fp32 [T, H]");
  fllm::TiedPrepareParams p{};
  const int64_t T = q_factor.size(0), H = q_factor.size(1), G = cache.size(1);
  TORCH_CHECK(i32(positions) && i32(slots) && positions.numel() >= T && slots.numel() >= T && k_offset >= H * dim && temp_every > 0, "positions, slots int32 [T]");
  if (splits > 0) {
    TORCH_CHECK(width >= k_offset + G * dim && given(q_out) && rows_of(*q_out, ty) && q_out->size(0) == T && q_out->size(1) >= H * dim, "q_out: [T, >= H * dim]");
    p.partials = partial_sums(workspace, splits, T, width);
    p.splits = (int)splits, p.width = (int)width, p.plane = T * width;
    p.q_out = q_out->data_ptr(), p.ld_qout = q_out->stride(0);
  } else {
    TORCH_CHECK(given(x) && rows_of(*x, ty) && x->size(0) == T && x->size(1) >= k_offset + G * dim, "x: [T, >= k_offset + G * dim]");
    p.x = x->data_ptr(), p.ldx = x->stride(0);
  }
  p.k_offset = (int)k_offset, p.H = (int)H, p.G = (int)G, p.dim = (int)dim, p.W = (int)cache.size(3), p.block_size = (int)cache.size(2), p.tokens = (int)T;
  p.positions = positions.data_ptr<int>(), p.slots = slots.data_ptr<int>();
  p.eps = (float)eps, p.scale = (float)scale, p.temp_coef = (float)temp_coef, p.temp_every = (float)temp_every;
  p.q_factor = q_factor.data_ptr<float>(), p.cache = cache.data_ptr(), p.key_factor = key_factor.data_ptr<float>();
  p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(cache.device());
  fllm::tied_prepare(p, cur_stream());
}

int64_t attention_tied_splits(int64_t num_seqs, int64_t max_q_len, int64_t H, int64_t G, int64_t max_kv_len) {
  return fllm::attention_tied_splits((int)num_seqs, (int)max_q_len, (int)H, (int)G, (int)max_kv_len);
}
int64_t attention_tied_workspace_bytes(int64_t tokens, int64_t H, int64_t W, int64_t splits) {
  return (int64_t)fllm::attention_tied_workspace_bytes((int)tokens, (int)H, (int)W, (int)splits);
}

// q [T, >= H * dim], out [T, >= H * dim]; returns the number of kernels launched
int64_t attention_tied(const Tensor& q, const Tensor& q_factor, const Tensor& cache, const Tensor& key_factor, int64_t dim, const Tensor& block_tables,
                       const Tensor& row_seq, const Tensor& positions, const Tensor& q_starts, Tensor out, int64_t num_seqs, int64_t max_q_len,
                       int64_t min_q_len, double softcap, int64_t splits, const optional<Tensor>& workspace, bool tensor_cores,
                       const optional<Tensor>& status) {
  const auto ty = act_type(q);
  TORCH_CHECK(rows_of(q, ty) && rows_of(out, ty) && f32(q_factor) && q_factor.dim() == 2 && q_factor.size(0) == q.size(0), "q, out: rows of one type; q_factor fp32 [T, H]");
  const int64_t T = q.size(0), H = q_factor.size(1);
  TORCH_CHECK(cache.dim() == 4 && cache.is_contiguous() && cache.scalar_type() == ty && f32(key_factor) && key_factor.numel() * cache.size(3) == cache.numel() &&
                  cache.size(3) >= dim && cache.size(1) > 0 && H % cache.size(1) == 0, "cache [blocks, heads, block_size, width], key_factor [blocks, heads, block_size]");
  TORCH_CHECK(q.size(1) >= H * dim && out.size(0) == T && out.size(1) >= H * dim, "q, out: [T, >= H * dim]");
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
  fllm::TiedAttnParams p{};
  p.q = q.data_ptr(), p.ldq = q.stride(0), p.q_factor = q_factor.data_ptr<float>(), p.cache = cache.data_ptr(), p.key_factor = key_factor.data_ptr<float>();
  p.block_tables = block_tables.data_ptr<int>(), p.max_blocks = (int)block_tables.stride(0);
  p.row_seq = row_seq.data_ptr<int>(), p.positions = positions.data_ptr<int>(), p.q_starts = q_starts.data_ptr<int>();
  p.out = out.data_ptr(), p.ldo = out.stride(0);
  p.tokens = (int)T, p.num_seqs = (int)num_seqs, p.max_q_len = (int)max_q_len, p.min_q_len = (int)min_q_len;
  p.H = (int)H, p.G = (int)cache.size(1), p.dim = (int)dim, p.W = (int)cache.size(3), p.block_size = (int)cache.size(2), p.num_blocks = cache.size(0);
  p.softcap = (float)softcap, p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(q.device());
  return fllm::attention_tied(p, (int)splits, ws, ws_bytes, tensor_cores, given(status) ? status->data_ptr<int>() : nullptr, cur_stream());
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("tied_prepare(Tensor? x, Tensor? workspace, int splits, int width, Tensor(a!)? q_out, int k_offset, int dim, Tensor positions, Tensor slots, "
        "float eps, float scale, float temp_coef, float temp_every, Tensor(b!) q_factor, Tensor(c!) cache, Tensor(d!) key_factor) -> ()", &tied_prepare);
  m.def("attention_tied_splits(int num_seqs, int max_q_len, int H, int G, int max_kv_len) -> int", &attention_tied_splits);
  m.def("attention_tied_workspace_bytes(int tokens, int H, int W, int splits) -> int", &attention_tied_workspace_bytes);
  m.def("attention_tied(Tensor q, Tensor q_factor, Tensor cache, Tensor key_factor, int dim, Tensor block_tables, Tensor row_seq, Tensor positions, "
        "Tensor q_starts, Tensor(a!) out, int num_seqs, int max_q_len, int min_q_len, float softcap, int splits, Tensor? workspace, bool tensor_cores, "
        "Tensor? status) -> int", &attention_tied);
}
