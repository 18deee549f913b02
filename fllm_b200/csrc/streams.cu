// Residual of several hyper-connected streams, kept in fp32: x [rows][S][ld]. A sublayer reads u = sum_s in[s] x_s through
// a norm and its output y comes back into every stream at once, x_t <- sum_s mix[s][t] x_s + out[t] y (mix is indexed
// [from][to]; a residual multiplier is folded into out). One kernel does the update behind a sublayer together with the
// read and the norm in front of the next one, so the streams cross memory once per sublayer: one read, one write. With
// S = 1 and unit coefficients this is an ordinary residual in fp32.
//
// The same kernel starts the streams (token ids instead of x: every stream is the embedding row) and ends them (in = 1:
// the sum of the streams through the final norm, only for the rows whose logits are wanted, nothing written back).
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
__device__ __forceinline__ void axpy(float4& a, float c, const float4& x) {
  a.x = fmaf(c, x.x, a.x), a.y = fmaf(c, x.y, a.y), a.z = fmaf(c, x.z, a.z), a.w = fmaf(c, x.w, a.w);
}

template <typename T>
struct StreamArgs {
  float* x;                    // [rows][S][ld]
  const int* ids;              // not null: the streams start as table[ids[row]]
  const T* table;
  int vocab;
  long long ld_table;
  const T* y;                  // sublayer output, null when the streams start
  long long ld_y;
  const float* partials;       // not null: y = sum over the splits of [splits][rows][ld] (a split-K projection's sums)
  int splits;
  long long plane;             // elements of one split
  const float *mix, *out, *in; // [S][S], [S], [S]
  const int* rows;             // not null: row r of the output reads row rows[r] of x and y
  const T *w, *b;              // norm weight and bias (b may be null), zero beyond `width`
  T* h;
  long long ld_h;
  int width, ld;               // values of a row, and its padded length (a multiple of 4; the padding stays zero)
  float eps;
  int rms, write;              // rms: x / sqrt(mean x^2 + eps) * w; otherwise the norm around the mean. write: store x
};

// block-wide sum; every thread gets it
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += red[i];
  return t;
}

template <typename T, int S, int ITERS>
__global__ void __launch_bounds__(512) stream_kernel(const StreamArgs<T> a) {
  __shared__ float red[16];
  __shared__ float coef[S * S + 2 * S];        // mix | out | in
  for (int i = threadIdx.x; i < S * S + 2 * S; i += blockDim.x) {
    float v = 0.f;
    if (i < S * S) v = a.mix ? a.mix[i] : 0.f;
    else if (i < S * S + S) v = a.out ? a.out[i - S * S] : 0.f;
    else v = a.in[i - S * S - S];
    coef[i] = v;
  }
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();
  const int row = a.rows ? a.rows[blockIdx.x] : (int)blockIdx.x;
  float* xr = a.x + (size_t)row * S * a.ld;
  const T* tr = nullptr;
  if (a.ids) {
    int id = a.ids[row];
    if (id < 0 || id >= a.vocab) id = 0;
    tr = a.table + (size_t)id * a.ld_table;
  }
  const int nvec = a.ld / 4;
  float4 u[ITERS];
  float sum = 0.f, sq = 0.f;
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int i = threadIdx.x + it * blockDim.x;
    u[it] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= nvec) continue;
    float4 n[S];
    if (a.ids) {
      const float4 e = load4(tr + 4 * i);
#pragma unroll
      for (int s = 0; s < S; ++s) n[s] = e;
    } else {
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
      float4 o[S];
#pragma unroll
      for (int s = 0; s < S; ++s) o[s] = load4(xr + (size_t)s * a.ld + 4 * i);
      if (a.partials) {
        const float* src = a.partials + (size_t)row * a.ld + 4 * i;
#pragma unroll 4
        for (int sp = 0; sp < a.splits; ++sp) {
          const float4 p = __ldcg(reinterpret_cast<const float4*>(src + sp * a.plane));
          y.x += p.x, y.y += p.y, y.z += p.z, y.w += p.w;
        }
      } else {
        y = load4(a.y + (size_t)row * a.ld_y + 4 * i);
      }
#pragma unroll
      for (int t = 0; t < S; ++t) {
        const float ot = coef[S * S + t];
        n[t] = make_float4(ot * y.x, ot * y.y, ot * y.z, ot * y.w);
#pragma unroll
        for (int s = 0; s < S; ++s) axpy(n[t], coef[s * S + t], o[s]);
      }
    }
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (a.write) store4(xr + (size_t)s * a.ld + 4 * i, n[s]);
      axpy(u[it], coef[S * S + S + s], n[s]);
    }
    sum += (u[it].x + u[it].y) + (u[it].z + u[it].w);            // the padding contributes zeros
  }
  float mean = 0.f;
  if (!a.rms) mean = block_sum(sum, red) / (float)a.width;
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int c = 4 * (threadIdx.x + it * blockDim.x);
    const float* v = &u[it].x;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (c + j < a.width) sq = fmaf(v[j] - mean, v[j] - mean, sq);
  }
  const float rstd = 1.f / sqrtf(block_sum(sq, red) / (float)a.width + a.eps);
  T* hr = a.h + (size_t)blockIdx.x * a.ld_h;
#pragma unroll
  for (int it = 0; it < ITERS; ++it) {
    const int i = threadIdx.x + it * blockDim.x;
    if (i >= nvec) continue;
    const float4 w = load4(a.w + 4 * i);
    float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
    if (a.b) b = load4(a.b + 4 * i);
    store4(hr + 4 * i, make_float4(fmaf((u[it].x - mean) * rstd, w.x, b.x), fmaf((u[it].y - mean) * rstd, w.y, b.y),
                                   fmaf((u[it].z - mean) * rstd, w.z, b.z), fmaf((u[it].w - mean) * rstd, w.w, b.w)));
  }
}

template <typename T, int S>
void launch_streams(const StreamArgs<T>& a, int rows, cudaStream_t s) {
  const int nvec = a.ld / 4;
  const int threads = std::min(512, (nvec + 31) / 32 * 32);
  const int iters = (nvec + threads - 1) / threads;
  if (iters <= 1) launch_pdl(stream_kernel<T, S, 1>, dim3(rows), dim3(threads), 0, s, a);
  else if (iters <= 2) launch_pdl(stream_kernel<T, S, 2>, dim3(rows), dim3(threads), 0, s, a);
  else if (iters <= 4) launch_pdl(stream_kernel<T, S, 4>, dim3(rows), dim3(threads), 0, s, a);
  else if (iters <= 8) launch_pdl(stream_kernel<T, S, 8>, dim3(rows), dim3(threads), 0, s, a);
  else throw std::runtime_error("stream_mix_norm: rows of at most 16384 values");
  cuda_check(cudaGetLastError(), "stream_kernel");
}

template <typename T>
void run_streams(const StreamMixParams& p, cudaStream_t s) {
  StreamArgs<T> a{p.x, p.ids, static_cast<const T*>(p.table), p.vocab, p.ld_table, static_cast<const T*>(p.y), p.ld_y, p.partials,
                  p.splits, p.plane, p.mix, p.out, p.in, p.rows, static_cast<const T*>(p.norm_w), static_cast<const T*>(p.norm_b),
                  static_cast<T*>(p.h), p.ld_h, p.width, p.ld, p.eps, p.rms, p.write};
  switch (p.streams) {
    case 1: return launch_streams<T, 1>(a, p.n_out, s);
    case 2: return launch_streams<T, 2>(a, p.n_out, s);
    case 3: return launch_streams<T, 3>(a, p.n_out, s);
    case 4: return launch_streams<T, 4>(a, p.n_out, s);
    case 5: return launch_streams<T, 5>(a, p.n_out, s);
    case 6: return launch_streams<T, 6>(a, p.n_out, s);
    case 7: return launch_streams<T, 7>(a, p.n_out, s);
    case 8: return launch_streams<T, 8>(a, p.n_out, s);
  }
  throw std::runtime_error("stream_mix_norm: 1 to 8 streams");
}
}  // namespace

void stream_mix_norm(const StreamMixParams& p, cudaStream_t s) {
  if (p.n_out <= 0) return;
  if ((p.ld & 3) || (p.ld_h & 3) || (p.ld_y & 3) || (p.ld_table & 3) || p.width > p.ld || p.width <= 0)
    throw std::runtime_error("stream_mix_norm: padded row lengths in multiples of 4");
  if (p.f32) run_streams<float>(p, s);
  else run_streams<bf16>(p, s);
}

}  // namespace fllm
