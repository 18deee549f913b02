// Device helpers of the recurrent kernels (recurrent.cu, recurrent_ssd.cu): element types, vector loads, state rows.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace fllm {
namespace {
using bf16 = __nv_bfloat16;

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + __expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(__expf(x)); }

// n consecutive bf16 values (n a multiple of 8, 16-byte aligned) widened into fp32 registers
template <int N>
__device__ __forceinline__ void load_bf16(const bf16* __restrict__ p, float (&out)[N]) {
  static_assert(N % 8 == 0, "slices are whole 16-byte words");
#pragma unroll
  for (int i = 0; i < N / 8; ++i) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p + 8 * i);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = __bfloat1622float2(h[j]);
      out[8 * i + 2 * j] = f.x;
      out[8 * i + 2 * j + 1] = f.y;
    }
  }
}
template <int N>
__device__ __forceinline__ void load_f32(const float* __restrict__ p, float (&out)[N]) {
#pragma unroll
  for (int i = 0; i < N / 4; ++i) {
    const float4 v = *reinterpret_cast<const float4*>(p + 4 * i);
    out[4 * i] = v.x, out[4 * i + 1] = v.y, out[4 * i + 2] = v.z, out[4 * i + 3] = v.w;
  }
}
template <int N>
__device__ __forceinline__ void store_f32(float* __restrict__ p, const float (&v)[N]) {
#pragma unroll
  for (int i = 0; i < N / 4; ++i)
    *reinterpret_cast<float4*>(p + 4 * i) = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
}
// element types of the kernels that also serve in 32-bit; fp32 activations take the accurate exponential
__device__ __forceinline__ float ld1(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float ld1(const float* p) { return *p; }
__device__ __forceinline__ void st1(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void st1(float* p, float v) { *p = v; }
__device__ __forceinline__ float2 ld2(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ void st2(bf16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }
__device__ __forceinline__ void st2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
template <typename T>
__device__ __forceinline__ float exp_t(float x) { return sizeof(T) == 4 ? expf(x) : __expf(x); }
template <typename T>
__device__ __forceinline__ float silu_t(float x) { return x / (1.f + exp_t<T>(-x)); }
template <typename T>
__device__ __forceinline__ float softplus_t(float x) { return x > 20.f ? x : log1pf(exp_t<T>(x)); }
template <int N>
__device__ __forceinline__ void load_row(const bf16* p, float (&out)[N]) { load_bf16<N>(p, out); }
template <int N>
__device__ __forceinline__ void load_row(const float* p, float (&out)[N]) { load_f32<N>(p, out); }
// the first n of N consecutive values, zeros behind them (any alignment)
template <int N, typename T>
__device__ __forceinline__ void load_part(const T* p, int n, float (&out)[N]) {
#pragma unroll
  for (int i = 0; i < N; ++i) out[i] = i < n ? ld1(p + i) : 0.f;
}
// sum over the LANES consecutive lanes that share one state row (LANES a power of two up to 32)
template <int LANES>
__device__ __forceinline__ float row_sum(float v) {
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// this lane's columns 4 (lk + TPK j) + 0..3 of a state row
template <int TPK, bool EXACT, int NPT>
__device__ __forceinline__ void load_state(const float* st, int lk, int DK, float (&S)[NPT]) {
#pragma unroll
  for (int j = 0; j < NPT / 4; ++j) {
    const int c = 4 * (lk + TPK * j);
    if (EXACT) {
      const float4 f = *reinterpret_cast<const float4*>(st + c);
      S[4 * j] = f.x, S[4 * j + 1] = f.y, S[4 * j + 2] = f.z, S[4 * j + 3] = f.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) S[4 * j + e] = c + e < DK ? st[c + e] : 0.f;
    }
  }
}
template <int TPK, bool EXACT, int NPT>
__device__ __forceinline__ void store_state(float* st, int lk, int DK, const float (&S)[NPT]) {
#pragma unroll
  for (int j = 0; j < NPT / 4; ++j) {
    const int c = 4 * (lk + TPK * j);
    if (EXACT) {
      *reinterpret_cast<float4*>(st + c) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < DK) st[c + e] = S[4 * j + e];
    }
  }
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
}  // namespace
}  // namespace fllm
