// True fp32 matrix products on the CUDA cores (no reduced-precision tensor mode), for models served in 32-bit:
// C[b][t][n] = sum_k A[b][t][k] B[b][n][k] (+ bias[n]) with arbitrary strides, so the same kernel is the linear layer
// (B = weight rows) and the batched per-head products. 64 x 64 tiles, 4 x 4 results per thread, K in steps of 16.
// Grouped form (mixture of experts): the row tiles come from a list built on the device, each with a matrix of its own.
#include <cuda_runtime.h>

#include <stdexcept>

#include "fllm_ops.h"
#include "tma_host.h"

namespace fllm {
namespace {
constexpr int TM = 64, TN = 64, TK = 16;

struct TileList {
  const int *expert, *row0, *count;
};

template <bool GROUPED>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32Params p, const TileList g) {
  __shared__ float As[TK][TM + 4], Bs[TK][TN + 4];
  if (GROUPED && (int)blockIdx.y >= *g.count) return;
  const int t0 = GROUPED ? g.row0[blockIdx.y] : blockIdx.y * TM, n0 = blockIdx.x * TN, tid = threadIdx.x;
  const float* A = p.a + (long long)blockIdx.z * p.a_b;
  const float* B = p.b + (long long)(GROUPED ? g.expert[blockIdx.y] : blockIdx.z) * p.b_b;
  const int tx = tid % 16, ty = tid / 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += TK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + i * 256;
      // neighbouring threads walk the operand's unit-stride dimension
      const int ak = p.a_k == 1 ? e % TK : e / TM, am = p.a_k == 1 ? e / TK : e % TM;
      As[ak][am] = (t0 + am < p.T && k0 + ak < p.K) ? A[(long long)(t0 + am) * p.a_t + (long long)(k0 + ak) * p.a_k] : 0.f;
      const int bk = p.b_k == 1 ? e % TK : e / TN, bn = p.b_k == 1 ? e / TK : e % TN;
      Bs[bk][bn] = (n0 + bn < p.N && k0 + bk < p.K) ? B[(long long)(n0 + bn) * p.b_n + (long long)(k0 + bk) * p.b_k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float av[4], bv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) av[i] = As[k][ty * 4 + i], bv[i] = Bs[k][tx + 16 * i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
  float* C = p.c + (long long)blockIdx.z * p.c_b;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + ty * 4 + i;
    if (t >= p.T) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      if (n < p.N) C[(long long)t * p.c_t + n] = acc[i][j] + (p.bias ? p.bias[n] : 0.f);
    }
  }
}
}  // namespace

void gemm_f32(const GemmF32Params& p, cudaStream_t s) {
  if (p.T <= 0 || p.N <= 0 || p.batch <= 0) return;
  if ((p.T + TM - 1) / TM > 65535 || p.batch > 65535) throw std::runtime_error("gemm_f32: too many rows for one launch");
  gemm_f32_kernel<false><<<dim3((p.N + TN - 1) / TN, (p.T + TM - 1) / TM, p.batch), 256, 0, s>>>(p, TileList{});
  cuda_check(cudaGetLastError(), "gemm_f32_kernel");
}

void moe_grouped_f32(const GemmF32Params& p, const int* tile_expert, const int* tile_row0, const int* num_tiles, int max_tiles, cudaStream_t s) {
  if (p.T <= 0 || p.N <= 0 || max_tiles <= 0) return;
  if (max_tiles > 65535) throw std::runtime_error("moe_grouped_f32: too many row tiles for one launch");
  gemm_f32_kernel<true><<<dim3((p.N + TN - 1) / TN, max_tiles, 1), 256, 0, s>>>(p, TileList{tile_expert, tile_row0, num_tiles});
  cuda_check(cudaGetLastError(), "moe_grouped_f32");
}

}  // namespace fllm
