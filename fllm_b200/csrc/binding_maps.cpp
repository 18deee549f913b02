// torch.ops.fllm_b200 bindings of attention of one or two maps over shared values (attention_maps.cu).
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
inline bool given(const optional<Tensor>& t) { return t.has_value() && t->defined(); }
inline bool i32(const Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous(); }
inline bool rows_of(const Tensor& t, at::ScalarType ty) { return t.is_cuda() && t.scalar_type() == ty && t.dim() == 2 && t.stride(1) == 1; }
inline at::ScalarType act_type(const Tensor& t) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat), "activations are bf16 or fp32 on a GPU");
  return t.scalar_type();
}
// key and value pools of one layer: [blocks, G * maps, block_size, wk] and [blocks, G, block_size, wv], maps 1 or 2
// (spread attention, `any`: one value row per token)
inline void check_pools(const Tensor& k, const Tensor& v, at::ScalarType ty, int64_t dim, int64_t v_dim, bool any = false) {
  TORCH_CHECK(k.dim() == 4 && v.dim() == 4 && k.is_contiguous() && v.is_contiguous() && k.is_cuda() && v.is_cuda() && k.scalar_type() == ty &&
                  v.scalar_type() == ty && k.size(0) == v.size(0) && k.size(2) == v.size(2) && k.size(3) >= dim && v.size(3) >= v_dim && dim > 0 && v_dim > 0 &&
                  (k.size(1) == v.size(1) || k.size(1) == 2 * v.size(1) || (any && v.size(1) == 1)),
              "pools: [blocks, heads (or twice as many), block_size, width] of one type");
}

// optional fp32 number per head
inline const float* per_head(const optional<Tensor>& t, int64_t H) {
  if (!given(t)) return nullptr;
  TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kFloat && t->is_contiguous() && t->numel() == H, "sinks and distance biases: fp32, one per query head");
  return t->data_ptr<float>();
}

// x [T, >= all segments], or its split-K partial sums [splits][T][width]; bias (optional) [width] is added. Norm weights (optional); eps < 0:
// no norms. conv_w [width, taps] with state rows [slots, taps - 1, width]: a causal convolution in front, every sequence has one token.
// extra_out [T, n]: columns from extra_offset on, as fp32.
void maps_prepare(const optional<Tensor>& x, const optional<Tensor>& workspace, int64_t splits, int64_t width, const optional<Tensor>& bias,
                  int64_t q_offset, int64_t k_offset, int64_t v_offset, int64_t dim, int64_t v_dim, const Tensor& positions, const Tensor& slots,
                  const Tensor& inv_freq, double rope_factor, bool pairs, const optional<Tensor>& q_norm, const optional<Tensor>& k_norm, bool full, double eps,
                  Tensor q_out, Tensor k_cache, Tensor v_cache, const optional<Tensor>& conv_w, const optional<Tensor>& conv_state,
                  const optional<Tensor>& seq_state, const optional<Tensor>& extra_out, int64_t extra_offset) {
  const auto ty = act_type(k_cache);
  check_pools(k_cache, v_cache, ty, dim, v_dim, true);
  TORCH_CHECK(q_out.is_cuda() && q_out.scalar_type() == ty && q_out.is_contiguous() && q_out.dim() == 3 && q_out.size(2) == k_cache.size(3),
              "q_out: [T, query maps, width of the key rows]");
  fllm::MapsPrepareParams p{};
  const int64_t T = q_out.size(0), HQ = q_out.size(1), HK = k_cache.size(1), G = v_cache.size(1);
  const int64_t end = std::max({q_offset + HQ * dim, k_offset + HK * dim, v_offset + G * v_dim});
  TORCH_CHECK(i32(positions) && i32(slots) && positions.numel() >= T && slots.numel() >= T && q_offset >= 0 && k_offset >= 0 && v_offset >= 0, "positions, slots int32 [T]");
  TORCH_CHECK(inv_freq.is_cuda() && inv_freq.scalar_type() == at::kFloat && inv_freq.is_contiguous() && 2 * inv_freq.numel() <= dim, "inv_freq: fp32, half the rotated values");
  if (given(q_norm)) {
    TORCH_CHECK(given(k_norm) && q_norm->is_cuda() && q_norm->scalar_type() == ty && q_norm->is_contiguous() && k_norm->is_cuda() && k_norm->scalar_type() == ty &&
                    k_norm->is_contiguous() && q_norm->numel() == (full ? HQ * dim : dim) && k_norm->numel() == (full ? HK * dim : dim),
                "norm weights: one map wide, or all maps (full)");
    p.q_norm = q_norm->data_ptr(), p.k_norm = k_norm->data_ptr();
  }
  if (given(conv_w)) {
    TORCH_CHECK(conv_w->is_cuda() && conv_w->scalar_type() == at::kFloat && conv_w->is_contiguous() && conv_w->dim() == 2 && conv_w->size(0) >= end &&
                    conv_w->size(1) >= 2 && given(conv_state) && conv_state->is_cuda() && conv_state->scalar_type() == ty && conv_state->is_contiguous() &&
                    conv_state->dim() == 3 && conv_state->size(1) == conv_w->size(1) - 1 && conv_state->size(2) == conv_w->size(0) && given(seq_state) &&
                    i32(*seq_state) && seq_state->numel() == T, "a convolution of single tokens: conv_w fp32 [width, taps], state [slots, taps - 1, width], one sequence per row");
    p.conv_w = conv_w->data_ptr<float>(), p.conv_state = conv_state->data_ptr(), p.seq_state = seq_state->data_ptr<int>();
    p.taps = (int)conv_w->size(1), p.conv_width = (int)conv_w->size(0);
  }
  if (splits > 0) {
    TORCH_CHECK(width >= end && given(workspace) && workspace->is_contiguous() && workspace->nbytes() >= fllm::kLinearPartialsOffset + (size_t)splits * T * width * 4,
                "workspace too small for the split-K partials");
    p.partials = reinterpret_cast<const float*>(reinterpret_cast<const uint8_t*>(workspace->data_ptr()) + fllm::kLinearPartialsOffset);
    p.splits = (int)splits, p.width = (int)width, p.plane = T * width;
  } else {
    TORCH_CHECK(given(x) && rows_of(*x, ty) && x->size(0) == T && x->size(1) >= end, "x: [T, >= all segments]");
    p.x = x->data_ptr(), p.ldx = x->stride(0);
  }
  if (given(extra_out)) {
    TORCH_CHECK(extra_out->is_cuda() && extra_out->scalar_type() == at::kFloat && extra_out->is_contiguous() && extra_out->dim() == 2 && extra_out->size(0) == T &&
                    extra_offset >= 0 && extra_offset + extra_out->size(1) <= (splits > 0 ? width : x->size(1)), "extra_out: fp32 [T, columns of the rows]");
    p.extra_out = extra_out->data_ptr<float>(), p.extra = (int)extra_out->size(1), p.extra_offset = (int)extra_offset;
  }
  if (given(bias)) {
    TORCH_CHECK(bias->is_cuda() && bias->scalar_type() == ty && bias->is_contiguous() && bias->numel() >= end, "bias: [width]");
    p.bias = bias->data_ptr();
  }
  p.q_offset = (int)q_offset, p.k_offset = (int)k_offset, p.v_offset = (int)v_offset, p.q_heads = (int)HQ, p.k_heads = (int)HK, p.v_heads = (int)G;
  p.dim = (int)dim, p.v_dim = (int)v_dim, p.wk = (int)k_cache.size(3), p.wv = (int)v_cache.size(3), p.block_size = (int)k_cache.size(2), p.tokens = (int)T;
  p.positions = positions.data_ptr<int>(), p.slots = slots.data_ptr<int>(), p.inv_freq = inv_freq.data_ptr<float>();
  p.rot = 2 * (int)inv_freq.numel(), p.rope_factor = (float)rope_factor, p.pairs = pairs ? 1 : 0;
  p.full = full ? 1 : 0, p.eps = (float)eps;
  p.q_out = q_out.data_ptr(), p.k_cache = k_cache.data_ptr(), p.v_cache = v_cache.data_ptr(), p.f32 = ty == at::kFloat ? 1 : 0;
  c10::cuda::CUDAGuard guard(k_cache.device());
  fllm::maps_prepare(p, cur_stream());
}

int64_t attention_maps_splits(int64_t num_seqs, int64_t max_q_len, int64_t H, int64_t G, int64_t maps, int64_t max_kv_len, int64_t window) {
  return fllm::attention_maps_splits((int)num_seqs, (int)max_q_len, (int)H, (int)G, (int)maps, (int)max_kv_len, (int)window);
}
int64_t attention_maps_workspace_bytes(int64_t tokens, int64_t q_heads, int64_t wv, int64_t splits) {
  return (int64_t)fllm::attention_maps_workspace_bytes((int)tokens, (int)q_heads, (int)wv, (int)splits);
}

// q [T, H * maps, wk], out [T, >= H * v_dim]; returns the number of kernels launched
int64_t attention_maps(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, int64_t dim, int64_t v_dim, const Tensor& block_tables,
                       const Tensor& row_seq, const Tensor& positions, const Tensor& q_starts, Tensor out, int64_t num_seqs, int64_t max_q_len,
                       int64_t min_q_len, double scale, int64_t window, double lam, double out_scale, double eps, int64_t splits,
                       const optional<Tensor>& workspace, bool tensor_cores, const optional<Tensor>& status, const optional<Tensor>& sink,
                       const optional<Tensor>& r1, const optional<Tensor>& r2) {
  const auto ty = act_type(q);
  check_pools(k_cache, v_cache, ty, dim, v_dim);
  const int64_t T = q.size(0), G = v_cache.size(1), M = k_cache.size(1) / G;
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && q.size(2) == k_cache.size(3) && q.size(1) % (G * M) == 0, "q: contiguous [T, H * maps, width of the key rows]");
  const int64_t H = q.size(1) / M;
  TORCH_CHECK(rows_of(out, ty) && out.size(0) == T && out.size(1) >= H * v_dim && window >= 0, "out: [T, >= H * v_dim] like q");
  TORCH_CHECK(block_tables.is_cuda() && block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 && block_tables.stride(1) == 1 && i32(row_seq) &&
                  i32(positions) && i32(q_starts) && row_seq.numel() >= T && positions.numel() >= T && q_starts.numel() >= num_seqs + 1,
              "block_tables [B, max_blocks], row_seq [T], positions [T], q_starts [B + 1]: int32");
  void* ws = nullptr;
  size_t ws_bytes = 0;
  if (given(workspace)) {
    TORCH_CHECK(workspace->is_cuda() && workspace->is_contiguous(), "workspace: contiguous CUDA tensor");
    ws = workspace->data_ptr();
    ws_bytes = workspace->nbytes();
  }
  fllm::MapsAttnParams p{};
  p.q = q.data_ptr(), p.k_cache = k_cache.data_ptr(), p.v_cache = v_cache.data_ptr();
  p.block_tables = block_tables.data_ptr<int>(), p.max_blocks = (int)block_tables.stride(0);
  p.row_seq = row_seq.data_ptr<int>(), p.positions = positions.data_ptr<int>(), p.q_starts = q_starts.data_ptr<int>();
  p.out = out.data_ptr(), p.ldo = out.stride(0);
  p.tokens = (int)T, p.num_seqs = (int)num_seqs, p.max_q_len = (int)max_q_len, p.min_q_len = (int)min_q_len;
  p.H = (int)H, p.G = (int)G, p.maps = (int)M, p.dim = (int)dim, p.v_dim = (int)v_dim, p.wk = (int)k_cache.size(3), p.wv = (int)v_cache.size(3);
  p.block_size = (int)k_cache.size(2), p.num_blocks = k_cache.size(0);
  p.scale = (float)scale, p.window = (int)window, p.lam = (float)lam, p.out_scale = (float)out_scale, p.eps = (float)eps, p.f32 = ty == at::kFloat ? 1 : 0;
  p.sink = per_head(sink, H), p.r1 = per_head(r1, H), p.r2 = per_head(r2, H);
  TORCH_CHECK((p.r1 != nullptr) == (p.r2 != nullptr), "a distance bias has two numbers per head");
  c10::cuda::CUDAGuard guard(q.device());
  return fllm::attention_maps(p, (int)splits, ws, ws_bytes, tensor_cores, given(status) ? status->data_ptr<int>() : nullptr, cur_stream());
}

// Talking heads: q [T, H, wk], value rows [blocks, 1, block_size, wv] with all heads' values (G * v_dim), talk fp32 [H, H], gate (optional) fp32
// [T, H] logits; part_o fp32 [T, H, splits, wv] and part_ml [T, H, splits, 2] are scratch. out [T, >= H * v_dim]. Returns the kernels launched.
int64_t attention_talk(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, int64_t dim, int64_t v_dim, const Tensor& block_tables,
                       const Tensor& row_seq, const Tensor& positions, const Tensor& q_starts, Tensor out, int64_t num_seqs, int64_t max_q_len,
                       int64_t min_q_len, double scale, int64_t window, const optional<Tensor>& sink, const optional<Tensor>& r1,
                       const optional<Tensor>& r2, const Tensor& talk, const optional<Tensor>& gate, Tensor part_o, Tensor part_ml, bool tensor_cores,
                       double bias_range, const optional<Tensor>& status) {
  const auto ty = act_type(q);
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4, "pools: [blocks, heads, block_size, width]");
  const int64_t T = q.size(0), G = k_cache.size(1), H = q.size(1), wv = v_cache.size(3);
  check_pools(k_cache, v_cache, ty, dim, G * v_dim, true);
  TORCH_CHECK(v_cache.size(1) == 1 && q.dim() == 3 && q.is_contiguous() && q.size(2) == k_cache.size(3) && H % G == 0, "q: contiguous [T, H, width of the key rows]");
  TORCH_CHECK(rows_of(out, ty) && out.size(0) == T && out.size(1) >= H * v_dim && window >= 0, "out: [T, >= H * v_dim] like q");
  TORCH_CHECK(block_tables.is_cuda() && block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 && block_tables.stride(1) == 1 && i32(row_seq) &&
                  i32(positions) && i32(q_starts) && row_seq.numel() >= T && positions.numel() >= T && q_starts.numel() >= num_seqs + 1,
              "block_tables [B, max_blocks], row_seq [T], positions [T], q_starts [B + 1]: int32");
  auto f32 = [](const Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous(); };
  TORCH_CHECK(f32(part_o) && part_o.dim() == 4 && part_o.size(0) == T && part_o.size(1) == H && part_o.size(3) == wv && f32(part_ml) &&
                  part_ml.numel() == T * H * part_o.size(2) * 2, "part_o fp32 [T, H, splits, wv], part_ml fp32 [T, H, splits, 2]");
  TORCH_CHECK(f32(talk) && talk.numel() == H * H && (!given(gate) || (rows_of(*gate, at::kFloat) && gate->size(0) == T && gate->size(1) >= H)),
              "talk fp32 [H, H], gate fp32 [T, H]");
  fllm::MapsAttnParams p{};
  p.q = q.data_ptr(), p.k_cache = k_cache.data_ptr(), p.v_cache = v_cache.data_ptr();
  p.block_tables = block_tables.data_ptr<int>(), p.max_blocks = (int)block_tables.stride(0);
  p.row_seq = row_seq.data_ptr<int>(), p.positions = positions.data_ptr<int>(), p.q_starts = q_starts.data_ptr<int>();
  p.tokens = (int)T, p.num_seqs = (int)num_seqs, p.max_q_len = (int)max_q_len, p.min_q_len = (int)min_q_len;
  p.H = (int)H, p.G = (int)G, p.maps = 1, p.dim = (int)dim, p.v_dim = (int)(G * v_dim), p.wk = (int)k_cache.size(3), p.wv = (int)wv;
  p.block_size = (int)k_cache.size(2), p.num_blocks = k_cache.size(0), p.scale = (float)scale, p.window = (int)window, p.f32 = ty == at::kFloat ? 1 : 0;
  p.r1 = per_head(r1, H), p.r2 = per_head(r2, H), p.spread = 1, p.part_o = part_o.data_ptr<float>(), p.part_ml = part_ml.data_ptr<float>();
  p.bias_range = (float)bias_range;
  TORCH_CHECK((p.r1 != nullptr) == (p.r2 != nullptr), "a distance bias has two numbers per head");
  fllm::TalkMixParams m{};
  m.part_o = p.part_o, m.part_ml = p.part_ml, m.sink = per_head(sink, H), m.talk = talk.data_ptr<float>();
  if (given(gate)) m.gate = gate->data_ptr<float>(), m.ld_gate = gate->stride(0);
  m.out = out.data_ptr(), m.ldo = out.stride(0), m.tokens = (int)T, m.H = (int)H, m.G = (int)G, m.splits = (int)part_o.size(2), m.v_dim = (int)v_dim;
  m.wv = (int)wv, m.cols = (int)out.size(1), m.f32 = p.f32;
  c10::cuda::CUDAGuard guard(q.device());
  const int n = fllm::attention_maps(p, m.splits, nullptr, 0, tensor_cores, given(status) ? status->data_ptr<int>() : nullptr, cur_stream());
  fllm::talk_mix(m, cur_stream());
  return n + 1;
}
int64_t attention_spread_splits(int64_t num_seqs, int64_t max_q_len, int64_t H, int64_t G, int64_t wv, int64_t max_kv_len, int64_t window) {
  return fllm::attention_spread_splits((int)num_seqs, (int)max_q_len, (int)H, (int)G, (int)wv, (int)max_kv_len, (int)window);
}
bool attention_spread_tc_supported(int64_t group, int64_t wk, int64_t wv, int64_t block_size) {
  return fllm::attention_spread_tc_supported((int)group, (int)wk, (int)wv, (int)block_size, 0);
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("maps_prepare(Tensor? x, Tensor? workspace, int splits, int width, Tensor? bias, int q_offset, int k_offset, int v_offset, int dim, int v_dim, "
        "Tensor positions, Tensor slots, Tensor inv_freq, float rope_factor, bool pairs, Tensor? q_norm, Tensor? k_norm, bool full, float eps, "
        "Tensor(a!) q_out, Tensor(b!) k_cache, Tensor(c!) v_cache, Tensor? conv_w, Tensor(d!)? conv_state, Tensor? seq_state, Tensor(e!)? extra_out, "
        "int extra_offset) -> ()", &maps_prepare);
  m.def("attention_maps_splits(int num_seqs, int max_q_len, int H, int G, int maps, int max_kv_len, int window) -> int", &attention_maps_splits);
  m.def("attention_maps_workspace_bytes(int tokens, int q_heads, int wv, int splits) -> int", &attention_maps_workspace_bytes);
  m.def("attention_maps(Tensor q, Tensor k_cache, Tensor v_cache, int dim, int v_dim, Tensor block_tables, Tensor row_seq, Tensor positions, Tensor q_starts, "
        "Tensor(a!) out, int num_seqs, int max_q_len, int min_q_len, float scale, int window, float lam, float out_scale, float eps, int splits, "
        "Tensor? workspace, bool tensor_cores, Tensor? status, Tensor? sink=None, Tensor? r1=None, Tensor? r2=None) -> int", &attention_maps);
  m.def("attention_spread_splits(int num_seqs, int max_q_len, int H, int G, int wv, int max_kv_len, int window) -> int", &attention_spread_splits);
  m.def("attention_spread_tc_supported(int group, int wk, int wv, int block_size) -> bool", &attention_spread_tc_supported);
  m.def("attention_talk(Tensor q, Tensor k_cache, Tensor v_cache, int dim, int v_dim, Tensor block_tables, Tensor row_seq, Tensor positions, Tensor q_starts, "
        "Tensor(a!) out, int num_seqs, int max_q_len, int min_q_len, float scale, int window, Tensor? sink, Tensor? r1, Tensor? r2, Tensor talk, Tensor? gate, "
        "Tensor(b!) part_o, Tensor(c!) part_ml, bool tensor_cores, float bias_range, Tensor? status) -> int", &attention_talk);
}
