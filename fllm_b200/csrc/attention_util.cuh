// Device helpers of the attention kernels over padded cache rows (attention_tied.cu, attention_maps.cu): element types, cp.async,
// ldmatrix and mma.sync wrappers of the decode kernels, the operand descriptor of values kept as [token][dim].
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <unordered_map>

#include "ptx.cuh"
#include "tma_host.h"

namespace fllm {
namespace {
using bf16 = __nv_bfloat16;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kPage = 16;                 // tokens fetched as one piece (blocks are multiples of it)

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// four consecutive values as one access
template <typename T>
struct Four { using type = uint2; };
template <>
struct Four<float> { using type = float4; };

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16-byte piece c of row r of a row-major tile lies at piece c ^ (r & 7): ldmatrix row fetches hit distinct banks
template <int D>
__device__ __forceinline__ bf16* tile_ptr(bf16* base, int row, int chunk) {
  return base + row * D + ((chunk ^ (row & 7)) << 3);
}

// tcgen05 tiles: 128 query rows or tokens; a 64-column half of one is kHalf bytes of 128-byte swizzled rows
constexpr int kRows = 128, kTile = 128, kHalf = 128 * 128;
constexpr float kLazyRescale = 8.f;
template <int D>
constexpr int tile_bytes() { return (D / 64) * kHalf; }

// MN-major operand: 128-byte swizzled rows, 1024 bytes between groups of eight rows, kHalf between the 64-column halves
template <int D>
__device__ __forceinline__ uint64_t desc_mn_major(uint32_t saddr) {
  return (uint64_t)((saddr & 0x3FFFFu) >> 4) | (uint64_t)((D > 64 ? kHalf : 1024) >> 4) << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}

// tensor map of a pool of `rows` rows of D values, in boxes of a page's rows and 64 columns
inline const CUtensorMap& pool_map(const void* pool, uint64_t rows, int D) {
  struct Key {
    const void* base;
    uint64_t rows;
    int d;
    bool operator==(const Key& o) const { return base == o.base && rows == o.rows && d == o.d; }
  };
  struct Hash {
    size_t operator()(const Key& k) const { return std::hash<const void*>()(k.base) ^ std::hash<uint64_t>()(k.rows * 2 + k.d / 128); }
  };
  static std::unordered_map<Key, CUtensorMap, Hash> maps;
  const Key key{pool, rows, D};
  auto it = maps.find(key);
  if (it == maps.end()) {
    if (maps.size() > 4096) maps.clear();
    it = maps.emplace(key, make_tmap_2d(pool, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, rows, D, D * 2, kPage, 64, true)).first;
  }
  return it->second;
}
}  // namespace
}  // namespace fllm
