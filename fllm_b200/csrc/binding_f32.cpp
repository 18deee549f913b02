// torch.ops.fllm_b200 bindings of the fp32 products (gemm_f32.cu).
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

// y = x @ w^T (+ bias), fp32
void linear_f32(const Tensor& x, const Tensor& w, const optional<Tensor>& bias, Tensor y) {
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == at::kFloat && w.scalar_type() == at::kFloat && y.scalar_type() == at::kFloat && x.dim() == 2 &&
                  w.dim() == 2 && y.dim() == 2 && y.stride(1) == 1 && x.size(1) == w.size(1) && y.size(0) == x.size(0) && y.size(1) == w.size(0),
              "linear_f32: x [T, K], w [N, K], y [T, N] in fp32");
  fllm::GemmF32Params p{};
  p.a = x.data_ptr<float>(), p.a_t = x.stride(0), p.a_k = x.stride(1);
  p.b = w.data_ptr<float>(), p.b_n = w.stride(0), p.b_k = w.stride(1);
  if (given(bias)) {
    TORCH_CHECK(bias->scalar_type() == at::kFloat && bias->is_contiguous() && bias->numel() == w.size(0), "linear_f32: bias");
    p.bias = bias->data_ptr<float>();
  }
  p.c = y.data_ptr<float>(), p.c_t = y.stride(0);
  p.batch = 1, p.T = (int)x.size(0), p.N = (int)w.size(0), p.K = (int)x.size(1);
  c10::cuda::CUDAGuard guard(x.device());
  fllm::gemm_f32(p, cur_stream());
}

// c[b] = a[b] @ m[b], fp32: a [B, T, K], m [B, K, N], c [B, T, N]
void bmm_f32(const Tensor& a, const Tensor& m, Tensor c) {
  TORCH_CHECK(a.is_cuda() && a.scalar_type() == at::kFloat && m.scalar_type() == at::kFloat && c.scalar_type() == at::kFloat && a.dim() == 3 &&
                  m.dim() == 3 && c.dim() == 3 && c.stride(2) == 1 && a.size(0) == m.size(0) && a.size(2) == m.size(1) && c.size(0) == a.size(0) &&
                  c.size(1) == a.size(1) && c.size(2) == m.size(2), "bmm_f32: a [B, T, K], m [B, K, N], c [B, T, N] in fp32");
  fllm::GemmF32Params p{};
  p.a = a.data_ptr<float>(), p.a_b = a.stride(0), p.a_t = a.stride(1), p.a_k = a.stride(2);
  p.b = m.data_ptr<float>(), p.b_b = m.stride(0), p.b_n = m.stride(2), p.b_k = m.stride(1);
  p.c = c.data_ptr<float>(), p.c_b = c.stride(0), p.c_t = c.stride(1);
  p.batch = (int)a.size(0), p.T = (int)a.size(1), p.N = (int)m.size(2), p.K = (int)a.size(2);
  c10::cuda::CUDAGuard guard(a.device());
  fllm::gemm_f32(p, cur_stream());
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(fllm_b200, m) {
  m.def("linear_f32(Tensor x, Tensor w, Tensor? bias, Tensor(a!) y) -> ()", &linear_f32);
  m.def("bmm_f32(Tensor a, Tensor m, Tensor(a!) c) -> ()", &bmm_f32);
}
