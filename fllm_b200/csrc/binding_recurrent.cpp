// torch.ops.fllm_b200 bindings of the recurrent token mixers (recurrent.cu, recurrent_ssd.cu, recurrent_chunk.cu).
#include <ATen/ATen.h>
#include <c10/cuda/CUDAGuard.h>
#include <c10/cuda/CUDAStream.h>
#include <torch/library.h>

#include "fllm_ops.h"

namespace {
using at::Tensor;
using c10::optional;
inline cudaStream_t cur_stream() { return c10::cuda::getCurrentCUDAStream().stream(); }
inline bool rows_bf16(const Tensor& t) { return t.is_cuda() && t.scalar_type() == at::kBFloat16 && t.dim() == 2 && t.stride(1) == 1; }
inline bool rows_of(const Tensor& t, at::ScalarType ty) { return t.is_cuda() && t.scalar_type() == ty && t.dim() == 2 && t.stride(1) == 1; }
// activation type of an op that exists in bf16 and in fp32
inline at::ScalarType act_type(const Tensor& t) {
  TORCH_CHECK(t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat, "activations are bf16 or fp32");
  return t.scalar_type();
}
inline const void* opt_ptr(const optional<Tensor>& t) { return t.has_value() && t->defined() ? t->data_ptr() : nullptr; }
inline const float* opt_f32(const optional<Tensor>& t) {
  if (!t.has_value() || !t->defined()) return nullptr;
  TORCH_CHECK(t->scalar_type() == at::kFloat && t->is_contiguous(), "parameter vectors are contiguous fp32");
  return t->data_ptr<float>();
}
inline long long opt_ld(const optional<Tensor>& t) { return t.has_value() && t->defined() ? t->stride(0) : 0; }
inline void check_batch(const Tensor& q_starts, const Tensor& seq_state, const Tensor& positions) {
  TORCH_CHECK(q_starts.scalar_type() == at::kInt && seq_state.scalar_type() == at::kInt && positions.scalar_type() == at::kInt &&
                  q_starts.is_contiguous() && seq_state.is_contiguous() && positions.is_contiguous() &&
                  q_starts.numel() == seq_state.numel() + 1,
              "q_starts [B + 1], seq_state [B], positions [T]: contiguous int32");
}

void causal_conv1d(const Tensor& x, const Tensor& w, const optional<Tensor>& bias, Tensor state, const Tensor& q_starts,
                   const Tensor& seq_state, const Tensor& positions, Tensor y, bool act, int64_t max_q_len) {
  const auto ty = act_type(x);
  TORCH_CHECK(rows_of(x, ty) && rows_of(y, ty) && x.sizes() == y.sizes(), "x, y: rows of one shape and type");
  const int64_t C = x.size(1), W = w.size(1);
  TORCH_CHECK(w.scalar_type() == at::kFloat && w.is_contiguous() && w.dim() == 2 && w.size(0) == C, "w: fp32 [C, W]");
  TORCH_CHECK(state.scalar_type() == ty && state.is_contiguous() && state.dim() == 3 && state.size(1) == W - 1 && state.size(2) == C,
              "state: [slots, W - 1, C] in the activation type");
  check_batch(q_starts, seq_state, positions);
  c10::cuda::CUDAGuard guard(x.device());
  const int rc = fllm::causal_conv1d(x.data_ptr(), x.stride(0), w.data_ptr<float>(), opt_f32(bias), state.data_ptr(), q_starts.data_ptr<int>(),
                                     seq_state.data_ptr<int>(), positions.data_ptr<int>(), y.data_ptr(), y.stride(0), (int)seq_state.numel(),
                                     (int)C, (int)W, act ? 1 : 0, (int)x.size(0), (int)(max_q_len > 0 ? max_q_len : x.size(0)), cur_stream(),
                                     ty == at::kFloat ? 1 : 0);
  TORCH_CHECK(rc == 0, "causal_conv1d: unsupported arguments (code ", rc, "): even C and strides, 2 <= W <= 8, y distinct from x");
}

void mamba2_scan(const Tensor& x, const Tensor& dt, const Tensor& Bm, const Tensor& Cm, const Tensor& A, const optional<Tensor>& D,
                 const optional<Tensor>& dt_bias, Tensor state, const Tensor& q_starts, const Tensor& seq_state, const Tensor& positions,
                 Tensor y, int64_t H, int64_t P, int64_t G, int64_t N, double dt_min, double dt_max, int64_t skip_from) {
  const auto ty = act_type(x);
  TORCH_CHECK(rows_of(x, ty) && rows_of(dt, ty) && rows_of(Bm, ty) && rows_of(Cm, ty) && rows_of(y, ty), "activations: rows of one type");
  TORCH_CHECK(x.size(1) == H * P && y.size(1) == H * P && dt.size(1) == H && Bm.size(1) == G * N && Cm.size(1) == G * N, "widths");
  TORCH_CHECK(state.scalar_type() == at::kFloat && state.is_contiguous() && state.dim() == 4 && state.size(1) == H && state.size(2) == P &&
                  state.size(3) == N, "state: fp32 [slots, H, P, N]");
  check_batch(q_starts, seq_state, positions);
  c10::cuda::CUDAGuard guard(x.device());
  fllm::SsdScanParams p{};
  p.x = x.data_ptr(), p.dt = dt.data_ptr(), p.Bm = Bm.data_ptr(), p.Cm = Cm.data_ptr();
  p.ldx = x.stride(0), p.lddt = dt.stride(0), p.ldb = Bm.stride(0), p.ldc = Cm.stride(0), p.ldy = y.stride(0);
  p.A = opt_f32(A), p.D = opt_f32(D), p.dt_bias = opt_f32(dt_bias), p.state = state.data_ptr<float>();
  p.q_starts = q_starts.data_ptr<int>(), p.seq_state = seq_state.data_ptr<int>(), p.positions = positions.data_ptr<int>(), p.y = y.data_ptr();
  p.B = (int)seq_state.numel(), p.tokens = (int)x.size(0), p.H = (int)H, p.P = (int)P, p.G = (int)G, p.N = (int)N;
  p.dt_min = (float)dt_min, p.dt_max = (float)dt_max, p.skip_from = (int)skip_from, p.f32 = ty == at::kFloat ? 1 : 0;
  const int rc = fllm::ssd_scan(p, cur_stream());
  TORCH_CHECK(rc == 0, "mamba2_scan: unsupported arguments (code ", rc, "): heads a multiple of the groups, state width up to 256");
}

// q, k [T, H * K], v, out [T, >= H * V], decay fp32 [H], state fp32 [slots, H, V, K]: S <- decay S + v' k'^T, out = S q'.
// chunked: q' = q (activations applied), the sequences with at least min_tokens tokens, over chunks on the tensor cores. Otherwise
// q' = silu(q), the sequences below skip_from (0: all), token by token.
void decay_scan(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& decay, Tensor state, const Tensor& q_starts,
                const Tensor& seq_state, const Tensor& positions, Tensor out, int64_t H, int64_t K, int64_t V, bool chunked, int64_t from, int64_t max_q_len) {
  const auto ty = act_type(v);
  TORCH_CHECK(rows_of(q, ty) && rows_of(k, ty) && rows_of(v, ty) && rows_of(out, ty), "activations: rows of one type");
  TORCH_CHECK(q.size(1) == H * K && k.size(1) == H * K && v.size(1) == H * V && out.size(1) >= H * V && out.size(0) == v.size(0) && decay.numel() == H, "widths");
  TORCH_CHECK(state.scalar_type() == at::kFloat && state.is_contiguous() && state.dim() == 4 && state.size(1) == H && state.size(2) == V &&
                  state.size(3) == K, "state: fp32 [slots, H, V, K]");
  check_batch(q_starts, seq_state, positions);
  c10::cuda::CUDAGuard guard(v.device());
  fllm::SsdScanParams p{};
  p.x = v.data_ptr(), p.Bm = k.data_ptr(), p.Cm = q.data_ptr();
  p.ldx = v.stride(0), p.ldb = k.stride(0), p.ldc = q.stride(0), p.ldy = out.stride(0);
  p.A = opt_f32(decay), p.state = state.data_ptr<float>();
  p.q_starts = q_starts.data_ptr<int>(), p.seq_state = seq_state.data_ptr<int>(), p.positions = positions.data_ptr<int>(), p.y = out.data_ptr();
  p.B = (int)seq_state.numel(), p.tokens = (int)v.size(0), p.H = (int)H, p.P = (int)V, p.G = (int)H, p.N = (int)K;
  p.f32 = ty == at::kFloat ? 1 : 0;
  p.skip_from = chunked ? 0 : (int)from;
  p.max_q_len = (int)max_q_len;
  const int rc = chunked ? fllm::decay_chunk(p, (int)from, cur_stream()) : fllm::ssd_scan(p, cur_stream());
  TORCH_CHECK(rc == 0, "decay_scan: unsupported arguments (code ", rc, "): key width up to 256; chunked: bf16, widths in multiples of 8, keys up to 128, aligned rows");
}

void mamba1_scan(const Tensor& x, const Tensor& dt, const Tensor& Bm, const Tensor& Cm, const optional<Tensor>& z, const Tensor& A,
                 const optional<Tensor>& D, const optional<Tensor>& dt_bias, Tensor state, const Tensor& q_starts, const Tensor& seq_state,
                 const Tensor& positions, Tensor y, int64_t seg_len, int64_t segs, const optional<Tensor>& seg_scratch) {
  TORCH_CHECK(rows_bf16(x) && rows_bf16(dt) && rows_bf16(Bm) && rows_bf16(Cm) && rows_bf16(y), "activations: bf16 rows");
  const int64_t Dm = x.size(1), N = Bm.size(1);
  TORCH_CHECK(A.scalar_type() == at::kFloat && A.is_contiguous() && A.dim() == 2 && A.size(0) == Dm && A.size(1) == N, "A: fp32 [D, N]");
  TORCH_CHECK(state.scalar_type() == at::kFloat && state.is_contiguous() && state.dim() == 3 && state.size(1) == Dm && state.size(2) == N,
              "state: fp32 [slots, D, N]");
  check_batch(q_starts, seq_state, positions);
  c10::cuda::CUDAGuard guard(x.device());
  float *seg_state = nullptr, *seg_dt = nullptr;
  const int64_t B = seq_state.numel();
  if (seg_len > 0 && segs > 1) {                 // scratch: B * segs states of [Dm][N], then [B][segs - 1][Dm] step sums
    const int64_t n_state = B * segs * Dm * N, n_dt = B * (segs - 1) * Dm;
    TORCH_CHECK(seg_scratch.has_value() && seg_scratch->scalar_type() == at::kFloat && seg_scratch->is_contiguous() &&
                    seg_scratch->numel() >= n_state + n_dt, "seg_scratch: fp32, at least B * Dm * (segs * N + segs - 1) values");
    seg_state = seg_scratch->data_ptr<float>();
    seg_dt = seg_state + n_state;
  }
  const int rc = fllm::mamba1_scan(x.data_ptr(), x.stride(0), dt.data_ptr(), dt.stride(0), Bm.data_ptr(), Bm.stride(0), Cm.data_ptr(),
                                   Cm.stride(0), opt_ptr(z), opt_ld(z), A.data_ptr<float>(), opt_f32(D), opt_f32(dt_bias),
                                   state.data_ptr<float>(), q_starts.data_ptr<int>(), seq_state.data_ptr<int>(), positions.data_ptr<int>(),
                                   y.data_ptr(), y.stride(0), (int)B, (int)Dm, (int)N, (int)seg_len, (int)segs, seg_state, seg_dt,
                                   cur_stream());
  TORCH_CHECK(rc == 0, "mamba1_scan: unsupported arguments (code ", rc, "): state width 8 / 16, B and C 16-byte aligned");
}

void matrix_state_scan(int64_t kind, const Tensor& r, const Tensor& k, const Tensor& v, const optional<Tensor>& a, const optional<Tensor>& b,
                       const optional<Tensor>& w_opt, const optional<Tensor>& u, const optional<Tensor>& beta, Tensor state, const Tensor& q_starts,
                       const Tensor& seq_state, const Tensor& positions, Tensor y, int64_t H, int64_t DK, int64_t DV, int64_t kv_ratio,
                       bool l2norm, double q_scale, const optional<Tensor>& gate_raw, const optional<Tensor>& gate_A,
                       const optional<Tensor>& gate_dt_bias) {
  const auto ty = act_type(r);
  TORCH_CHECK(rows_of(r, ty) && rows_of(k, ty) && rows_of(v, ty) && rows_of(y, ty), "activations: rows of one type");
  TORCH_CHECK(v.size(1) == H * DV && y.size(1) == H * DV && r.size(1) == (H / kv_ratio) * DK && k.size(1) == r.size(1), "widths");
  const bool raw = !(w_opt.has_value() && w_opt->defined());
  const float* w_ptr = nullptr;
  long long w_ld = 0;
  if (!raw) {
    const Tensor& w = *w_opt;
    TORCH_CHECK(w.is_cuda() && w.scalar_type() == at::kFloat && w.dim() == 2 && w.stride(1) == 1, "w: fp32 rows of log decays");
    TORCH_CHECK(w.size(1) == (kind == 2 ? H : r.size(1)), "w: one decay per head (kind 2) or per key channel");
    w_ptr = w.data_ptr<float>();
    w_ld = w.stride(0);
  } else {
    TORCH_CHECK(kind == 2 && gate_raw.has_value() && rows_of(*gate_raw, ty) && gate_raw->size(1) == H && gate_A.has_value() &&
                    gate_dt_bias.has_value() && gate_A->numel() == H && gate_dt_bias->numel() == H,
                "raw gates: kind 2 with gate_raw [T, H], gate_A and gate_dt_bias fp32 [H]");
  }
  TORCH_CHECK(kind != 1 || (a.has_value() && b.has_value() && rows_bf16(*a) && rows_bf16(*b)), "RWKV-7 needs a and b");
  TORCH_CHECK(kind != 0 || (u.has_value() && u->numel() == r.size(1)), "RWKV-6 needs the bonus u");
  TORCH_CHECK(kind < 2 || (beta.has_value() && rows_of(*beta, ty) && beta->size(1) == H), "delta rules need beta [T, H]");
  TORCH_CHECK(state.scalar_type() == at::kFloat && state.is_contiguous() && state.dim() == 4 && state.size(1) == H && state.size(2) == DV &&
                  state.size(3) == DK, "state: fp32 [slots, H, DV, DK]");
  check_batch(q_starts, seq_state, positions);
  c10::cuda::CUDAGuard guard(r.device());
  const int rc = fllm::matrix_state_scan((int)kind, r.data_ptr(), r.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), opt_ptr(a),
                                         opt_ld(a), opt_ptr(b), opt_ld(b), w_ptr, w_ld, opt_f32(u), opt_ptr(beta),
                                         opt_ld(beta), state.data_ptr<float>(), q_starts.data_ptr<int>(), seq_state.data_ptr<int>(),
                                         positions.data_ptr<int>(), y.data_ptr(), y.stride(0), (int)seq_state.numel(), (int)H, (int)DK, (int)DV,
                                         (int)kv_ratio, l2norm ? 1 : 0, (float)q_scale, opt_ptr(gate_raw), opt_ld(gate_raw), opt_f32(gate_A),
                                         opt_f32(gate_dt_bias), (int)r.size(0), cur_stream(), ty == at::kFloat ? 1 : 0);
  TORCH_CHECK(rc == 0, "matrix_state_scan: unsupported arguments (code ", rc, "): key width up to 256 (kind 2), 32 / 64 / 128 / 256 with 16-byte aligned bf16 rows (other kinds)");
}

void gated_rmsnorm(const Tensor& x, const optional<Tensor>& z, const Tensor& w, Tensor y, int64_t group_size, double eps, bool norm_before_gate,
                   bool sigmoid_gate) {
  const auto ty = act_type(x);
  TORCH_CHECK(rows_of(x, ty) && rows_of(y, ty) && x.sizes() == y.sizes(), "x, y: rows of one shape and type");
  TORCH_CHECK(w.scalar_type() == ty && w.is_contiguous() && x.size(1) % group_size == 0, "w: like x; D a multiple of the group");
  TORCH_CHECK(!z.has_value() || !z->defined() || (rows_of(*z, ty) && z->sizes() == x.sizes()), "z: rows like x");
  c10::cuda::CUDAGuard guard(x.device());
  fllm::gated_rmsnorm(x.data_ptr(), x.stride(0), opt_ptr(z), opt_ld(z), w.data_ptr(), (int)w.numel(), y.data_ptr(), y.stride(0), (int)x.size(0),
                      (int)x.size(1), (int)group_size, (float)eps, norm_before_gate ? 1 : 0, cur_stream(), ty == at::kFloat ? 1 : 0, sigmoid_gate ? 1 : 0);
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("causal_conv1d(Tensor x, Tensor w, Tensor? bias, Tensor(a!) state, Tensor q_starts, Tensor seq_state, Tensor positions, Tensor(b!) y, bool act, int max_q_len) -> ()",
        &causal_conv1d);
  m.def("mamba2_scan(Tensor x, Tensor dt, Tensor Bm, Tensor Cm, Tensor A, Tensor? D, Tensor? dt_bias, Tensor(a!) state, Tensor q_starts, "
        "Tensor seq_state, Tensor positions, Tensor(b!) y, int H, int P, int G, int N, float dt_min, float dt_max, int skip_from) -> ()",
        &mamba2_scan);
  m.def("decay_scan(Tensor q, Tensor k, Tensor v, Tensor decay, Tensor(a!) state, Tensor q_starts, Tensor seq_state, Tensor positions, Tensor(b!) out, "
        "int H, int K, int V, bool chunked, int from_tokens, int max_q_len) -> ()", &decay_scan);
  m.def("mamba1_scan(Tensor x, Tensor dt, Tensor Bm, Tensor Cm, Tensor? z, Tensor A, Tensor? D, Tensor? dt_bias, Tensor(a!) state, "
        "Tensor q_starts, Tensor seq_state, Tensor positions, Tensor(b!) y, int seg_len, int segs, Tensor? seg_scratch) -> ()",
        &mamba1_scan);
  m.def("matrix_state_scan(int kind, Tensor r, Tensor k, Tensor v, Tensor? a, Tensor? b, Tensor? w, Tensor? u, Tensor? beta, Tensor(a!) state, "
        "Tensor q_starts, Tensor seq_state, Tensor positions, Tensor(b!) y, int H, int DK, int DV, int kv_ratio, bool l2norm, float q_scale, "
        "Tensor? gate_raw, Tensor? gate_A, Tensor? gate_dt_bias) -> ()",
        &matrix_state_scan);
  m.def("gated_rmsnorm(Tensor x, Tensor? z, Tensor w, Tensor(a!) y, int group_size, float eps, bool norm_before_gate, bool sigmoid_gate=False) -> ()", &gated_rmsnorm);
}
