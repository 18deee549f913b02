// Residual in fp32 with the norm in front of a sublayer. One kernel covers every place where the residual x [rows][ld] changes:
//   start    x = table[id]
//   update   x' = x + y (+ table[id])            y: the output of the sublayer behind it, or the split-K partial sums of its projection
// and what the next sublayer reads goes out in the activation type: h = x' / sqrt(mean x'^2 + eps) * (w_offset + w), and with a token
// shift h_t + (h_(t-1) - h_t) mu, where h_(t-1) is the normalised row of the sequence's token before (zeros in front of the first).
//
// With a token shift a CTA takes a few consecutive rows and computes the row in front of them once more, so x' goes to a buffer of
// its own. The normalised row of a sequence's last token is kept in a state row (fp32); the CTA with the sequence's first row in a
// step both reads and writes it, computing the last row as well where that row belongs to another CTA.
#include <cuda_bf16.h>

#include <algorithm>
#include <stdexcept>

#include "fllm_ops.h"
#include "ptx.cuh"
#include "tma_host.h"

namespace fllm {
namespace {
using bf16 = __nv_bfloat16;

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ float4 plus(const float4& a, const float4& b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 zero4() { return make_float4(0.f, 0.f, 0.f, 0.f); }

// the new residual of one row
template <typename T, int ITERS>
__device__ __forceinline__ void new_row(const PreNormParams& p, int row, float4 (&v)[ITERS]) {
  const int nvec = p.ld / 4;
  const T* tr = nullptr;
  if (p.ids) {
    int id = p.ids[row];
    if (id < 0 || id >= p.vocab) id = 0;
    tr = static_cast<const T*>(p.table) + (size_t)id * p.ld_table;
  }
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int i = threadIdx.x + it * blockDim.x;
    v[it] = zero4();
    if (i >= nvec) continue;
    if (p.x) v[it] = load4(p.x + (size_t)row * p.ld + 4 * i);
    if (p.partials) {
      const float* src = p.partials + (size_t)row * p.ld + 4 * i;
      float4 y = zero4();
#pragma unroll 4
      for (int sp = 0; sp < p.splits; ++sp) y = plus(y, __ldcg(reinterpret_cast<const float4*>(src + sp * p.plane)));
      v[it] = plus(v[it], y);
    } else if (p.y) {
      v[it] = plus(v[it], load4(static_cast<const T*>(p.y) + (size_t)row * p.ld_y + 4 * i));
    }
    if (tr) v[it] = plus(v[it], load4(tr + 4 * i));
  }
}

// v -> its norm (the padding is zero and stays zero)
template <int ITERS>
__device__ __forceinline__ void normalise(const PreNormParams& p, const float4 (&w)[ITERS], float4 (&v)[ITERS], float* red) {
  float sq = 0.f;
#pragma unroll
  for (int it = 0; it < ITERS; ++it) sq += fmaf(v[it].x, v[it].x, v[it].y * v[it].y) + fmaf(v[it].z, v[it].z, v[it].w * v[it].w);
  sq = warp_sum(sq);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += red[i];
  const float r = 1.f / sqrtf(t / (float)p.width + p.eps);
#pragma unroll
  for (int it = 0; it < ITERS; ++it) v[it] = make_float4(v[it].x * r * w[it].x, v[it].y * r * w[it].y, v[it].z * r * w[it].z, v[it].w * r * w[it].w);
}

template <typename T, int ITERS, bool SHIFT>
__global__ void __launch_bounds__(512) prenorm_kernel(const PreNormParams p) {
  __shared__ float red[16];
  const int nvec = p.ld / 4;
  pdl_launch_dependents();
  float4 w[ITERS];
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {           // weights do not wait for the kernel before
    const int i = threadIdx.x + it * blockDim.x;
    w[it] = zero4();
    if (i < nvec) {
      w[it] = load4(static_cast<const T*>(p.norm_w) + 4 * i);
      w[it] = make_float4(p.w_offset + w[it].x, p.w_offset + w[it].y, p.w_offset + w[it].z, p.w_offset + w[it].w);
    }
  }
  pdl_wait();
  T* h = static_cast<T*>(p.h);
  if (!SHIFT) {
    const int row = p.rows ? p.rows[blockIdx.x] : (int)blockIdx.x;
    float4 v[ITERS];
    new_row<T, ITERS>(p, row, v);
    if (p.x_out) {
#pragma unroll
      for (int it = 0; it < ITERS; ++it) {
        const int i = threadIdx.x + it * blockDim.x;
        if (i < nvec) store4(p.x_out + (size_t)row * p.ld + 4 * i, v[it]);
      }
    }
    normalise<ITERS>(p, w, v, red);
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int i = threadIdx.x + it * blockDim.x;
      if (i < nvec) store4(h + (size_t)blockIdx.x * p.ld_h + 4 * i, v[it]);
    }
    return;
  }
  const int lo = blockIdx.x * p.rows_per, hi = min(lo + p.rows_per, p.n_out);
  float4 prev[ITERS];
  for (int row = lo; row < hi; ++row) {
    const int seq = p.single ? row : p.row_seq[row], first = p.q_starts[seq], last = p.q_starts[seq + 1] - 1;
    float* state = p.state + (size_t)p.seq_state[seq] * p.ld;
    if (row == first) {
      const bool fresh = p.positions[row] == 0;
#pragma unroll
      for (int it = 0; it < ITERS; ++it) {
        const int i = threadIdx.x + it * blockDim.x;
        prev[it] = !fresh && i < nvec ? load4(state + 4 * i) : zero4();
      }
      if (last >= hi) {                            // the sequence ends in another CTA: its last row is computed here too
        float4 v[ITERS];
        new_row<T, ITERS>(p, last, v);
        normalise<ITERS>(p, w, v, red);
#pragma unroll
        for (int it = 0; it < ITERS; ++it) {
          const int i = threadIdx.x + it * blockDim.x;
          if (i < nvec) store4(state + 4 * i, v[it]);
        }
      }
    } else if (row == lo) {
      new_row<T, ITERS>(p, row - 1, prev);
      normalise<ITERS>(p, w, prev, red);
    }
    float4 v[ITERS];
    new_row<T, ITERS>(p, row, v);
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int i = threadIdx.x + it * blockDim.x;
      if (i < nvec) store4(p.x_out + (size_t)row * p.ld + 4 * i, v[it]);
    }
    normalise<ITERS>(p, w, v, red);
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int i = threadIdx.x + it * blockDim.x;
      if (i < nvec) {
        const float4 m = load4(static_cast<const T*>(p.shift) + 4 * i);
        store4(h + (size_t)row * p.ld_h + 4 * i, make_float4(fmaf(prev[it].x - v[it].x, m.x, v[it].x), fmaf(prev[it].y - v[it].y, m.y, v[it].y),
                                                             fmaf(prev[it].z - v[it].z, m.z, v[it].z), fmaf(prev[it].w - v[it].w, m.w, v[it].w)));
        if (row == last && first >= lo) store4(state + 4 * i, v[it]);
      }
      prev[it] = v[it];
    }
  }
}

template <typename T, bool SHIFT>
void run(const PreNormParams& p, int ctas, cudaStream_t s) {
  const int nvec = p.ld / 4, threads = std::min(512, (nvec + 31) / 32 * 32), iters = (nvec + threads - 1) / threads;
  const dim3 grid(ctas), block(threads);
  if (iters <= 1) launch_pdl(prenorm_kernel<T, 1, SHIFT>, grid, block, 0, s, p);
  else if (iters <= 2) launch_pdl(prenorm_kernel<T, 2, SHIFT>, grid, block, 0, s, p);
  else if (iters <= 4) launch_pdl(prenorm_kernel<T, 4, SHIFT>, grid, block, 0, s, p);
  else if (iters <= 8) launch_pdl(prenorm_kernel<T, 8, SHIFT>, grid, block, 0, s, p);
  else throw std::runtime_error("prenorm: rows of at most 16384 values");
  cuda_check(cudaGetLastError(), "prenorm_kernel");
}
}  // namespace

void prenorm(const PreNormParams& params, cudaStream_t s) {
  PreNormParams p = params;
  if (p.n_out <= 0) return;
  if ((p.ld & 3) || (p.ld_h & 3) || (p.ld_y & 3) || (p.ld_table & 3) || p.width > p.ld || p.width <= 0)
    throw std::runtime_error("prenorm: padded row lengths in multiples of 4");
  if (p.shift == nullptr) {
    if (p.f32) run<float, false>(p, p.n_out, s);
    else run<bf16, false>(p, p.n_out, s);
    return;
  }
  if (p.rows || !p.x_out || p.x == p.x_out) throw std::runtime_error("prenorm: a token shift needs every row and a residual buffer of its own to write");
  // one row in `rows_per` is computed twice; few rows go one per CTA
  p.rows_per = p.single || p.n_out <= 4 * sm_count() ? 1 : std::min(8, (p.n_out + 4 * sm_count() - 1) / (4 * sm_count()));
  const int ctas = (p.n_out + p.rows_per - 1) / p.rows_per;
  if (p.f32) run<float, true>(p, ctas, s);
  else run<bf16, true>(p, ctas, s);
}

}  // namespace fllm
