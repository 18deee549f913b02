// Residual in fp32 whose norm comes after the sum, and the per-layer token input. One kernel covers every place where the
// residual x [rows][ld] changes, with y the output of the sublayer behind it (or the split-K partial sums of its projection):
//   start      x = table[id] * scale
//   norm sum   x <- rms(alpha x + y) w                 a block whose norm follows the residual sum
//   add norm   x <- x + rms(y) w                       an output that is normalised before it is added
// where rms(v) = v / sqrt(mean v^2 + eps). y may itself be half the sum of two projections, each normalised with a weight of its
// own (PAIR): y = (rms(a) wa + rms(b) wb) / 2. Behind it the row goes on to the next projection, rounded to the activation type, or
// through a second RMS norm (times a factor) in front of the head, then only for the rows whose logits are wanted.
//
// side_gate: g = gelu_tanh(gate) * e with e a slice of the token's row in a table of per-layer embeddings.
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
__device__ __forceinline__ float dot4(const float4& v) { return fmaf(v.x, v.x, v.y * v.y) + fmaf(v.z, v.z, v.w * v.w); }
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += red[i];
  return t;
}

__device__ __forceinline__ float2 block_sum2(float a, float b, float2* red) {
  a = warp_sum(a), b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(a, b);
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t.x += red[i].x, t.y += red[i].y;
  return t;
}

template <typename T, int ITERS, bool PAIR>
__global__ void __launch_bounds__(512) postnorm_kernel(const PostNormParams p) {
  __shared__ float red[16];
  pdl_launch_dependents();
  pdl_wait();
  const int row = p.rows ? p.rows[blockIdx.x] : (int)blockIdx.x;
  float* xr = p.x + (size_t)row * p.ld;
  const int nvec = p.ld / 4;
  float4 v[ITERS];
  if (p.ids) {
    int id = p.ids[row];
    if (id < 0 || id >= p.vocab) id = 0;
    const T* tr = static_cast<const T*>(p.table) + (size_t)id * p.ld_table;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int i = threadIdx.x + it * blockDim.x;
      if (i >= nvec) continue;
      const float4 e = load4(tr + 4 * i);
      v[it] = make_float4(e.x * p.scale, e.y * p.scale, e.z * p.scale, e.w * p.scale);
    }
  } else {
    float4 x[ITERS], a[PAIR ? ITERS : 1];
    float sq = 0.f, sqa = 0.f;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int i = threadIdx.x + it * blockDim.x;
      v[it] = x[it] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i >= nvec) continue;
      x[it] = load4(xr + 4 * i);
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
      if (p.partials) {
        const float* src = p.partials + (size_t)row * p.ld + 4 * i;
#pragma unroll 4
        for (int sp = 0; sp < p.splits; ++sp) {
          const float4 q = __ldcg(reinterpret_cast<const float4*>(src + sp * p.plane));
          y.x += q.x, y.y += q.y, y.z += q.z, y.w += q.w;
        }
      } else {
        y = load4(static_cast<const T*>(p.y) + (size_t)row * p.ld_y + 4 * i);
      }
      if constexpr (PAIR) {
        v[it] = y;
        a[it] = load4(static_cast<const T*>(p.pair_a) + (size_t)row * p.ld_pair + 4 * i);
        sqa += dot4(a[it]), sq += dot4(y);
        continue;
      }
      if (!p.add) y = make_float4(fmaf(p.alpha, x[it].x, y.x), fmaf(p.alpha, x[it].y, y.y), fmaf(p.alpha, x[it].z, y.z), fmaf(p.alpha, x[it].w, y.w));
      v[it] = y;
      sq += dot4(y);                                       // the padding is zero
    }
    if constexpr (PAIR) {
      __shared__ float2 red2[16];
      const float2 s2 = block_sum2(sqa, sq, red2);
      const float ra = 0.5f / sqrtf(s2.x / (float)p.width + p.eps), rb = 0.5f / sqrtf(s2.y / (float)p.width + p.eps);
      sq = 0.f;
#pragma unroll
      for (int it = 0; it < ITERS; ++it) {
        const int i = threadIdx.x + it * blockDim.x;
        if (i >= nvec) continue;
        const float4 wa = load4(static_cast<const T*>(p.pair_wa) + 4 * i), wb = load4(static_cast<const T*>(p.pair_wb) + 4 * i);
        float4 y = make_float4(fmaf(a[it].x * ra, wa.x, v[it].x * rb * wb.x), fmaf(a[it].y * ra, wa.y, v[it].y * rb * wb.y),
                               fmaf(a[it].z * ra, wa.z, v[it].z * rb * wb.z), fmaf(a[it].w * ra, wa.w, v[it].w * rb * wb.w));
        if (!p.add) y = make_float4(fmaf(p.alpha, x[it].x, y.x), fmaf(p.alpha, x[it].y, y.y), fmaf(p.alpha, x[it].z, y.z), fmaf(p.alpha, x[it].w, y.w));
        v[it] = y;
        sq += dot4(y);
      }
    }
    const float r = 1.f / sqrtf(block_sum(sq, red) / (float)p.width + p.eps);
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int i = threadIdx.x + it * blockDim.x;
      if (i >= nvec) continue;
      const float4 w = load4(static_cast<const T*>(p.norm_w) + 4 * i);
      const float4 b = p.add ? x[it] : make_float4(0.f, 0.f, 0.f, 0.f);
      v[it] = make_float4(fmaf(v[it].x * r, w.x, b.x), fmaf(v[it].y * r, w.y, b.y), fmaf(v[it].z * r, w.z, b.z), fmaf(v[it].w * r, w.w, b.w));
    }
  }
  if (p.write) {
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int i = threadIdx.x + it * blockDim.x;
      if (i < nvec) store4(xr + 4 * i, v[it]);
    }
  }
  T* hr = static_cast<T*>(p.h) + (size_t)blockIdx.x * p.ld_h;
  if (p.final_w == nullptr) {
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
      const int i = threadIdx.x + it * blockDim.x;
      if (i < nvec) store4(hr + 4 * i, v[it]);
    }
    return;
  }
  float sq = 0.f;
#pragma unroll
  for (int it = 0; it < ITERS; ++it)
    if ((int)(threadIdx.x + it * blockDim.x) < nvec) sq += dot4(v[it]);
  const float r = p.final_scale / sqrtf(block_sum(sq, red) / (float)p.width + p.eps);
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int i = threadIdx.x + it * blockDim.x;
    if (i >= nvec) continue;
    const float4 w = load4(static_cast<const T*>(p.final_w) + 4 * i);
    store4(hr + 4 * i, make_float4(v[it].x * r * w.x, v[it].y * r * w.y, v[it].z * r * w.z, v[it].w * r * w.w));
  }
}

template <typename T, bool PAIR>
void run_postnorm(const PostNormParams& p, cudaStream_t s) {
  const int nvec = p.ld / 4, threads = std::min(512, (nvec + 31) / 32 * 32), iters = (nvec + threads - 1) / threads;
  const dim3 grid(p.n_out), block(threads);
  if (iters <= 1) launch_pdl(postnorm_kernel<T, 1, PAIR>, grid, block, 0, s, p);
  else if (iters <= 2) launch_pdl(postnorm_kernel<T, 2, PAIR>, grid, block, 0, s, p);
  else if (iters <= 4) launch_pdl(postnorm_kernel<T, 4, PAIR>, grid, block, 0, s, p);
  else if (iters <= 8) launch_pdl(postnorm_kernel<T, 8, PAIR>, grid, block, 0, s, p);
  else throw std::runtime_error("postnorm: rows of at most 16384 values");
  cuda_check(cudaGetLastError(), "postnorm_kernel");
}

// columns [dim, cols) of the output are zero
template <typename T>
__global__ void __launch_bounds__(256) side_gate_kernel(const SideGateParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const long long item = (long long)blockIdx.x * 256 + threadIdx.x;
  const int t = (int)(item / p.cols), c = (int)(item % p.cols);
  if (t >= p.tokens) return;
  float v = 0.f;
  if (c < p.dim) {
    float z = 0.f;
    if (p.partials) {
      const float* src = p.partials + (size_t)t * p.cols + c;
      for (int sp = 0; sp < p.splits; ++sp) z += __ldcg(src + sp * p.plane);
    } else {
      z = to_f32(static_cast<const T*>(p.gate)[(long long)t * p.ld_gate + c]);
    }
    int id = p.ids[t];
    if (id < 0 || id >= p.vocab) id = 0;
    const float e = to_f32(static_cast<const T*>(p.table)[(long long)id * p.ld_table + p.offset + c]);
    v = 0.5f * z * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z))) * e;
  }
  put(static_cast<T*>(p.out) + (long long)t * p.ld_out + c, v);
}
}  // namespace

void postnorm(const PostNormParams& p, cudaStream_t s) {
  if (p.n_out <= 0) return;
  if ((p.ld & 3) || (p.ld_h & 3) || (p.ld_y & 3) || (p.ld_table & 3) || p.width > p.ld || p.width <= 0)
    throw std::runtime_error("postnorm: padded row lengths in multiples of 4");
  if (p.pair_a != nullptr) {
    if (p.ld_pair & 3) throw std::runtime_error("postnorm: padded row lengths in multiples of 4");
    if (p.f32) run_postnorm<float, true>(p, s);
    else run_postnorm<bf16, true>(p, s);
    return;
  }
  if (p.f32) run_postnorm<float, false>(p, s);
  else run_postnorm<bf16, false>(p, s);
}

void side_gate(const SideGateParams& p, cudaStream_t s) {
  if (p.tokens <= 0) return;
  const dim3 grid((unsigned)(((long long)p.tokens * p.cols + 255) / 256));
  if (p.f32) launch_pdl(side_gate_kernel<float>, grid, dim3(256), 0, s, p);
  else launch_pdl(side_gate_kernel<bf16>, grid, dim3(256), 0, s, p);
  cuda_check(cudaGetLastError(), "side_gate_kernel");
}

}  // namespace fllm
