// torch.ops.fllm_b200 bindings of the attention kernels over a paged K / V pool and of the 576-wide latent attention.
#include <ATen/ATen.h>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <c10/cuda/CUDAStream.h>
#include <torch/library.h>

#include "fllm_ops.h"

namespace {

using at::Tensor;
using c10::optional;

inline cudaStream_t cur_stream() { return c10::cuda::getCurrentCUDAStream().stream(); }

inline void check_bf16(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == at::kBFloat16, name, " must be bfloat16");
}
inline void check_i32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == at::kInt, name, " must be int32");
  TORCH_CHECK(t.is_contiguous(), name, " must be contiguous");
}
inline void check_rows(const Tensor& t, const char* name) {
  TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1, name, " must be 2-D with a unit inner stride");
}
template <typename T>
inline const T* opt_ptr(const optional<Tensor>& t) {
  return t.has_value() && t->defined() ? reinterpret_cast<const T*>(t->data_ptr()) : nullptr;
}

inline bool rows_bf16(const Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kBFloat16 && t.dim() == 2 && t.stride(1) == 1; }

void attention_generic(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache,
                       const Tensor& block_tables, const Tensor& row_seq, const Tensor& positions,
                       Tensor out, int64_t hq, int64_t hkv, int64_t head_dim, double scale,
                       int64_t window, const optional<Tensor>& sinks, double softcap,
                       const optional<Tensor>& tree_mask, const optional<Tensor>& tree_base) {
  check_bf16(q, "q"); check_rows(q, "q"); check_bf16(out, "out"); check_rows(out, "out");
  check_i32(block_tables, "block_tables"); check_i32(row_seq, "row_seq");
  check_i32(positions, "positions");
  const unsigned long long* tm = nullptr;
  const int* tb = nullptr;
  if (tree_mask.has_value() && tree_mask->defined()) {        // draft trees: one 64-bit ancestor mask and one context length per row
    TORCH_CHECK(tree_base.has_value() && tree_base->defined(), "attention_generic: tree_mask needs tree_base");
    TORCH_CHECK(tree_mask->scalar_type() == at::kLong && tree_mask->is_contiguous() && tree_mask->numel() == q.size(0), "tree_mask: int64 [rows]");
    check_i32(*tree_base, "tree_base");
    TORCH_CHECK(tree_base->numel() == q.size(0), "tree_base: int32 [rows]");
    tm = reinterpret_cast<const unsigned long long*>(tree_mask->data_ptr<int64_t>());
    tb = tree_base->data_ptr<int>();
  }
  const bool kv_fp8 = k_cache.element_size() == 1;            // e4m3 bytes instead of bf16
  TORCH_CHECK(k_cache.is_cuda() && k_cache.is_contiguous() && v_cache.is_contiguous() &&
              k_cache.element_size() == v_cache.element_size() && (kv_fp8 || k_cache.scalar_type() == at::kBFloat16),
              "caches must be contiguous bf16 or 1-byte e4m3 tensors");
  c10::cuda::CUDAGuard guard(q.device());
  fllm::attention_generic_bf16(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(),
                               block_tables.data_ptr<int>(), (int)block_tables.size(1),
                               row_seq.data_ptr<int>(), positions.data_ptr<int>(), out.data_ptr(),
                               out.stride(0), (int)q.size(0), (int)hq, (int)hkv, (int)head_dim,
                               (int)k_cache.size(2), (float)scale, (int)window,
                               opt_ptr<float>(sinks), (float)softcap, cur_stream(), kv_fp8 ? 1 : 0, tm, tb);
}

int64_t attention_tc(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache,
                     const Tensor& block_tables, const Tensor& q_starts, const Tensor& kv_lens, Tensor out,
                     int64_t num_seqs, int64_t max_q_len, int64_t min_q_len, int64_t max_kv_len, int64_t hq,
                     int64_t hkv, int64_t head_dim, double scale, int64_t window,
                     const optional<Tensor>& sinks, double softcap, const optional<Tensor>& workspace,
                     const optional<Tensor>& status, bool bidirectional) {
  check_bf16(q, "q"); check_rows(q, "q"); check_bf16(out, "out"); check_rows(out, "out");
  const bool kv_fp8 = k_cache.element_size() == 1;            // e4m3 bytes: the decode kernel widens them to f16
  TORCH_CHECK(k_cache.is_cuda() && v_cache.is_cuda() && k_cache.is_contiguous() && v_cache.is_contiguous() &&
              k_cache.element_size() == v_cache.element_size() && (kv_fp8 || k_cache.scalar_type() == at::kBFloat16),
              "caches must be contiguous bf16 or 1-byte e4m3 tensors");
  check_i32(q_starts, "q_starts"); check_i32(kv_lens, "kv_lens");
  TORCH_CHECK(block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 &&
              block_tables.stride(1) == 1 && block_tables.stride(0) == block_tables.size(1),
              "block_tables must be a dense int32 matrix");
  TORCH_CHECK(q_starts.numel() >= num_seqs + 1 && kv_lens.numel() >= num_seqs, "attention_tc: metadata too short");
  c10::cuda::CUDAGuard guard(q.device());
  void* ws = nullptr;
  size_t ws_bytes = 0;
  if (workspace.has_value() && workspace->defined()) { ws = workspace->data_ptr(); ws_bytes = workspace->nbytes(); }
  return fllm::attention_tc_bf16(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(),
                                 block_tables.data_ptr<int>(), (int)block_tables.size(1),
                                 q_starts.data_ptr<int>(), kv_lens.data_ptr<int>(), out.data_ptr(),
                                 out.stride(0), (int)q.size(0), (int)num_seqs, (int)max_q_len,
                                 (int)min_q_len, (int)max_kv_len, (int)hq, (int)hkv, (int)head_dim,
                                 (int)k_cache.size(2), (float)scale, (int)window, opt_ptr<float>(sinks),
                                 (float)softcap, ws, ws_bytes, cur_stream(), (long long)k_cache.size(0),
                                 const_cast<int*>(opt_ptr<int>(status)), kv_fp8 ? 1 : 0, bidirectional ? 1 : 0);
}

// q_abs [H, T, 512] or [T, H, 512] (any strides with a unit inner one), q_pe [T, H, 64], out like q_abs
int64_t attention_mla_splits(int64_t tokens, int64_t H, int64_t max_kv_len) {
  return fllm::attention_mla_splits((int)tokens, (int)H, (int)max_kv_len);
}
int64_t attention_mla_workspace_bytes(int64_t tokens, int64_t H, int64_t splits) {
  return (int64_t)fllm::attention_mla_workspace_bytes((int)tokens, (int)H, (int)splits);
}

// splits = 0: the CUDA-core kernel; >= 1: the tensor-core kernel over that many key slices (workspace needed above 1)
void attention_mla(const Tensor& q_abs, const Tensor& q_pe, const Tensor& cache, const Tensor& block_tables, const Tensor& row_seq,
                   const Tensor& positions, Tensor out, bool head_major, double scale, int64_t splits, const optional<Tensor>& workspace) {
  TORCH_CHECK(q_abs.is_cuda() && q_abs.scalar_type() == at::kBFloat16 && q_abs.dim() == 3 && q_abs.stride(2) == 1 && q_abs.size(2) == 512,
              "q_abs: bf16 [., ., 512] with a unit inner stride");
  TORCH_CHECK(out.scalar_type() == at::kBFloat16 && out.dim() == 3 && out.stride(2) == 1 && out.sizes() == q_abs.sizes(), "out: like q_abs");
  const int td = head_major ? 1 : 0, hd = head_major ? 0 : 1;
  const int64_t T = q_abs.size(td), H = q_abs.size(hd);
  TORCH_CHECK(q_pe.scalar_type() == at::kBFloat16 && q_pe.is_contiguous() && q_pe.dim() == 3 && q_pe.size(0) == T && q_pe.size(1) == H &&
                  q_pe.size(2) == 64, "q_pe: contiguous bf16 [T, H, 64]");
  TORCH_CHECK(cache.scalar_type() == at::kBFloat16 && cache.dim() == 3 && cache.is_contiguous() && cache.size(2) == 576,
              "cache: contiguous bf16 [blocks, block_size, 576]");
  TORCH_CHECK(block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 && block_tables.stride(1) == 1 &&
                  row_seq.scalar_type() == at::kInt && positions.scalar_type() == at::kInt && row_seq.is_contiguous() &&
                  positions.is_contiguous() && row_seq.numel() >= T && positions.numel() >= T,
              "block_tables [B, max_blocks], row_seq [T], positions [T]: int32");
  c10::cuda::CUDAGuard guard(q_abs.device());
  if (splits >= 1) {
    void* ws = nullptr;
    size_t ws_bytes = 0;
    if (workspace.has_value() && workspace->defined()) {
      TORCH_CHECK(workspace->is_cuda() && workspace->is_contiguous(), "workspace: contiguous CUDA tensor");
      ws = workspace->data_ptr();
      ws_bytes = workspace->numel() * workspace->element_size();
    }
    fllm::attention_mla_tc_bf16(q_abs.data_ptr(), q_abs.stride(td), q_abs.stride(hd), q_pe.data_ptr(), cache.data_ptr(),
                                block_tables.data_ptr<int>(), (int)block_tables.stride(0), row_seq.data_ptr<int>(), positions.data_ptr<int>(),
                                out.data_ptr(), out.stride(td), out.stride(hd), (int)T, (int)H, (int)cache.size(1), (float)scale, (int)splits,
                                ws, ws_bytes, cur_stream());
    return;
  }
  fllm::attention_mla_bf16(q_abs.data_ptr(), q_abs.stride(td), q_abs.stride(hd), q_pe.data_ptr(), cache.data_ptr(), block_tables.data_ptr<int>(),
                           (int)block_tables.stride(0), row_seq.data_ptr<int>(), positions.data_ptr<int>(), out.data_ptr(), out.stride(td),
                           out.stride(hd), (int)T, (int)H, (int)cache.size(1), (float)scale, cur_stream());
}

// ckv bf16 [T, >= 576] rows, q bf16 [T, H, head] contiguous with the rotary values of a head at rope_offset
void mla_prepare(const Tensor& ckv, const Tensor& q, int64_t rope_offset, const Tensor& positions, const Tensor& slots, const Tensor& inv_freq,
                 double attn_factor, const Tensor& norm_w, double eps, Tensor cache, Tensor q_pe) {
  TORCH_CHECK(rows_bf16(ckv) && ckv.size(1) >= 576, "ckv: bf16 rows of at least 576 values");
  TORCH_CHECK(q.is_cuda() && q.scalar_type() == at::kBFloat16 && q.dim() == 3 && q.is_contiguous() && rope_offset + 64 <= q.size(2) &&
                  q.size(0) == ckv.size(0), "q: contiguous bf16 [T, H, head]");
  TORCH_CHECK(inv_freq.scalar_type() == at::kFloat && inv_freq.is_contiguous() && inv_freq.numel() == 32, "inv_freq: fp32 [32]");
  TORCH_CHECK(norm_w.scalar_type() == at::kBFloat16 && norm_w.is_contiguous() && norm_w.numel() == 512, "norm_w: bf16 [512]");
  TORCH_CHECK(cache.scalar_type() == at::kBFloat16 && cache.is_contiguous() && cache.dim() == 3 && cache.size(2) == 576, "cache: bf16 [blocks, block_size, 576]");
  TORCH_CHECK(q_pe.scalar_type() == at::kBFloat16 && q_pe.is_contiguous() && q_pe.dim() == 3 && q_pe.size(0) == q.size(0) &&
                  q_pe.size(1) == q.size(1) && q_pe.size(2) == 64, "q_pe: contiguous bf16 [T, H, 64]");
  TORCH_CHECK(positions.scalar_type() == at::kInt && slots.scalar_type() == at::kInt && positions.is_contiguous() && slots.is_contiguous() &&
                  positions.numel() >= q.size(0) && slots.numel() >= q.size(0), "positions, slots: int32 [T]");
  c10::cuda::CUDAGuard guard(q.device());
  fllm::mla_prepare_bf16(ckv.data_ptr(), ckv.stride(0), q.data_ptr(), q.stride(0), (int)q.stride(1), (int)rope_offset, positions.data_ptr<int>(),
                         slots.data_ptr<int>(), inv_freq.data_ptr<float>(), (float)attn_factor, norm_w.data_ptr(), (float)eps, cache.data_ptr(),
                         q_pe.data_ptr(), (int)q.size(0), (int)q.size(1), cur_stream());
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("attention_generic(Tensor q, Tensor k_cache, Tensor v_cache, Tensor block_tables, Tensor row_seq, Tensor positions, Tensor(a!) out, int hq, int hkv, int head_dim, float scale, int window, Tensor? sinks, float softcap, Tensor? tree_mask=None, Tensor? tree_base=None) -> ()", &attention_generic);
  m.def("attention_tc(Tensor q, Tensor k_cache, Tensor v_cache, Tensor block_tables, Tensor q_starts, Tensor kv_lens, Tensor(a!) out, int num_seqs, int max_q_len, int min_q_len, int max_kv_len, int hq, int hkv, int head_dim, float scale, int window, Tensor? sinks, float softcap, Tensor? workspace, Tensor? status=None, bool bidirectional=False) -> int", &attention_tc);
  m.def("attention_mla(Tensor q_abs, Tensor q_pe, Tensor cache, Tensor block_tables, Tensor row_seq, Tensor positions, Tensor(a!) out, "
        "bool head_major, float scale, int splits, Tensor? workspace) -> ()", &attention_mla);
  m.def("attention_mla_splits(int tokens, int H, int max_kv_len) -> int", &attention_mla_splits);
  m.def("attention_mla_workspace_bytes(int tokens, int H, int splits) -> int", &attention_mla_workspace_bytes);
  m.def("mla_prepare(Tensor ckv, Tensor q, int rope_offset, Tensor positions, Tensor slots, Tensor inv_freq, float attn_factor, Tensor norm_w, "
        "float eps, Tensor(a!) cache, Tensor(b!) q_pe) -> ()", &mla_prepare);
}
