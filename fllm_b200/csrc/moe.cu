// Mixture-of-experts routing and data movement around the grouped tcgen05 GEMM:
//
//   moe_route_kernel    one warp per token: top-k over the router logits, weights = softmax over
//                       the selected logits (gpt-oss) or softmax over all experts renormalised
//                       over the selection (Mixtral / Qwen-MoE);
//   moe_align_kernel    one CTA: count rows per expert, lay the experts' row segments out back to
//                       back, each padded to the token-tile width, and emit the tile list
//                       (expert, first row) that the grouped GEMM walks; sizes stay on the device
//                       so the whole layer can live in a CUDA graph; optionally each row's routing
//                       weight;
//   moe_gather_kernel   permuted activations xp[row] = x[token(row)] (zero rows for padding);
//   moe_combine_kernel  out[token] = sum_j weight[token, j] * y[row(token, j)] in slot order, so
//                       the result does not depend on scheduling.
//
// Reference counterparts: rust/engine/cuda/moe.cu:40-150 (moe_route2), :159-205 (moe_align),
// :533-597 (combine2). The reference routes on the host inside a device group
// (rust/engine/src/rust_decoder.rs:7621-7729); here nothing leaves the device.
#include <algorithm>

#include "fllm_ops.h"
#include "ptx.cuh"
#include "tma_host.h"

namespace fllm {

__global__ void moe_route_kernel(const __nv_bfloat16* __restrict__ logits, long long ld, const __nv_bfloat16* __restrict__ bias,
                                 int tokens, int experts, int k, int softmax_all, int* __restrict__ ids,
                                 float* __restrict__ weights) {
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= tokens) return;
  constexpr int MAXPL = 8;                      // up to 256 experts
  float v[MAXPL];
#pragma unroll
  for (int i = 0; i < MAXPL; ++i) {
    const int e = lane + 32 * i;
    v[i] = e < experts ? __bfloat162float(logits[(size_t)t * ld + e]) + (bias ? __bfloat162float(bias[e]) : 0.f) : -INFINITY;
  }
  float denom_all = 0.f, vmax = -INFINITY;
  if (softmax_all) {
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) vmax = fmaxf(vmax, v[i]);
    vmax = warp_max(vmax);
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) denom_all += v[i] == -INFINITY ? 0.f : __expf(v[i] - vmax);
    denom_all = warp_sum(denom_all);
  }
  float sel_v[8];
  int sel_e[8];
  // a logit that is not a number counts as -inf, and a winner is marked as taken: the k experts are valid and distinct whatever comes in
  unsigned open = 0;
#pragma unroll
  for (int i = 0; i < MAXPL; ++i) {
    if (v[i] != v[i]) v[i] = -INFINITY;
    open |= lane + 32 * i < experts ? 1u << i : 0u;
  }
  for (int j = 0; j < k; ++j) {
    float best = -INFINITY;
    int best_e = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) {
      const int e = lane + 32 * i;
      if ((open >> i & 1) && (v[i] > best || (v[i] == best && e < best_e))) { best = v[i]; best_e = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, best_e, o);
      if (ob > best || (ob == best && oe < best_e)) { best = ob; best_e = oe; }
    }
    sel_v[j] = best;
    sel_e[j] = best_e;
    if ((best_e & 31) == lane) open &= ~(1u << (best_e >> 5));    // remove the winner
  }
  if (lane == 0) {
    float w[8], sum = 0.f;
    for (int j = 0; j < k; ++j) {
      w[j] = softmax_all ? __expf(sel_v[j] - vmax) / denom_all : __expf(sel_v[j] - sel_v[0]);
      sum += w[j];
    }
    for (int j = 0; j < k; ++j) {
      ids[(size_t)t * k + j] = sel_e[j];
      weights[(size_t)t * k + j] = w[j] / sum;
    }
  }
}

// Routers that weigh experts by their score: score = softmax over all experts (score_kind 1) or sigmoid (2) of the logit; the
// k experts with the largest score + select_bias are taken (the bias only steers the choice: DeepSeek-V3, GLM-4.5, ERNIE 4.5);
// weights = the scores of the chosen experts, renormalised on request, times `scale`. With groups of neighbouring experts only the
// experts of the best groups (by their best choice score) can be taken. One warp per token, up to 256 experts.
// Logits: bf16, or (Sum) fp32 as the sum of planes, then with the accurate exponential.
struct Bf16Logits {
  const __nv_bfloat16* p;
  long long ld;
  static constexpr bool kAccurate = false;
  __device__ __forceinline__ float operator()(int t, int e) const { return __bfloat162float(p[(size_t)t * ld + e]); }
};
struct SumLogits {
  const float* p;
  long long ld, plane;
  int splits;
  static constexpr bool kAccurate = true;
  __device__ __forceinline__ float operator()(int t, int e) const {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) v += __ldcg(p + s * plane + (size_t)t * ld + e);
    return v;
  }
};
template <typename Logits>
__global__ void moe_route_scored_kernel(const Logits logits, const float* __restrict__ select_bias, int tokens, int experts, int k,
                                        int score_kind, int renorm, float scale, const RouteGroups gr, int* __restrict__ ids,
                                        float* __restrict__ weights, float* __restrict__ gate_out) {
  __shared__ float choice[4][256], best_of[4][256];
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= tokens) return;
  constexpr int MAXPL = 8;
  auto ex = [](float x) { return Logits::kAccurate ? expf(x) : __expf(x); };
  float sc[MAXPL], ch[MAXPL];
  float vmax = -INFINITY;
#pragma unroll
  for (int i = 0; i < MAXPL; ++i) {
    const int e = lane + 32 * i;
    sc[i] = e < experts ? logits(t, e) : -INFINITY;
    vmax = fmaxf(vmax, sc[i]);
  }
  if (score_kind == 1) {
    vmax = warp_max(vmax);
    float den = 0.f;
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) {
      sc[i] = sc[i] == -INFINITY ? 0.f : ex(sc[i] - vmax);
      den += sc[i];
    }
    den = warp_sum(den);
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) sc[i] /= den;
  } else {
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) sc[i] = sc[i] == -INFINITY ? 0.f : 1.f / (1.f + ex(-sc[i]));
  }
#pragma unroll
  for (int i = 0; i < MAXPL; ++i) {
    const int e = lane + 32 * i;
    ch[i] = e < experts ? sc[i] + (select_bias ? select_bias[e] : 0.f) : -INFINITY;
  }
  if (gr.groups > 1) {
    float* mine = choice[threadIdx.x >> 5];
    float* group = best_of[threadIdx.x >> 5];
    const int per = experts / gr.groups;
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) mine[lane + 32 * i] = ch[i];
    __syncwarp();
    for (int g = lane; g < gr.groups; g += 32) {
      float m = -INFINITY;
      for (int e = g * per; e < (g + 1) * per; ++e) m = fmaxf(m, mine[e]);
      group[g] = m;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) {
      const int e = lane + 32 * i;
      if (e >= experts) continue;
      const int g = e / per;
      const float own = group[g];
      int ahead = 0;
      for (int o = 0; o < gr.groups; ++o) ahead += group[o] > own || (group[o] == own && o < g);
      if (ahead >= gr.keep) ch[i] = gr.masked;
    }
  }
  if (gate_out != nullptr && lane == 0) gate_out[t] = 1.f / (1.f + ex(-logits(t, experts)));
  float sel_s[8];
  int sel_e[8];
  unsigned open = 0;      // as in moe_route_kernel: valid and distinct experts whatever the scores are
#pragma unroll
  for (int i = 0; i < MAXPL; ++i) {
    if (ch[i] != ch[i]) ch[i] = -INFINITY;
    open |= lane + 32 * i < experts ? 1u << i : 0u;
  }
  for (int j = 0; j < k; ++j) {
    float best = -INFINITY, best_s = 0.f;
    int best_e = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < MAXPL; ++i) {
      const int e = lane + 32 * i;
      if ((open >> i & 1) && (ch[i] > best || (ch[i] == best && e < best_e))) { best = ch[i]; best_e = e; best_s = sc[i]; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o), os = __shfl_xor_sync(0xffffffffu, best_s, o);
      const int oe = __shfl_xor_sync(0xffffffffu, best_e, o);
      if (ob > best || (ob == best && oe < best_e)) { best = ob; best_e = oe; best_s = os; }
    }
    sel_s[j] = best_s;
    sel_e[j] = best_e;
    if ((best_e & 31) == lane) open &= ~(1u << (best_e >> 5));    // remove the winner
  }
  if (lane == 0) {
    float sum = 0.f;
    for (int j = 0; j < k; ++j) sum += sel_s[j];
    const float f = (renorm ? 1.f / (sum + 1e-20f) : 1.f) * scale;
    for (int j = 0; j < k; ++j) {
      ids[(size_t)t * k + j] = sel_e[j];
      weights[(size_t)t * k + j] = sel_s[j] * f;
    }
  }
}

void moe_route_scored(const void* logits, long long ld, const float* select_bias, int tokens, int experts, int k, int score_kind,
                      int renorm, float scale, int* ids, float* weights, cudaStream_t s) {
  if (tokens <= 0) return;
  if (experts > 256 || k > 8 || k > experts || (score_kind != 1 && score_kind != 2)) throw std::runtime_error("moe_route_scored: at most 256 experts, top-8, score kind 1 or 2");
  moe_route_scored_kernel<<<(tokens + 3) / 4, 128, 0, s>>>(Bf16Logits{(const __nv_bfloat16*)logits, ld}, select_bias, tokens, experts, k,
                                                           score_kind, renorm, scale, RouteGroups{}, ids, weights, (float*)nullptr);
  cuda_check(cudaGetLastError(), "moe_route_scored_kernel");
}

void moe_route_fp32(const float* logits, int splits, long long plane, long long ld, int tokens, int experts, int k, int score_kind, int renorm,
                    float scale, int* ids, float* weights, cudaStream_t s, const float* select_bias, const RouteGroups& groups, float* gate_out) {
  if (tokens <= 0) return;
  if (experts > 256 || k > 8 || k > experts || (score_kind != 1 && score_kind != 2)) throw std::runtime_error("moe_route_fp32: at most 256 experts, top-8, score kind 1 or 2");
  if (groups.groups < 1 || experts % groups.groups || groups.keep < 1) throw std::runtime_error("moe_route_fp32: equal groups of experts");
  moe_route_scored_kernel<<<(tokens + 3) / 4, 128, 0, s>>>(SumLogits{logits, ld, plane, splits}, select_bias, tokens, experts, k, score_kind,
                                                           renorm, scale, groups, ids, weights, gate_out);
  cuda_check(cudaGetLastError(), "moe_route_fp32");
}

void moe_route(const void* logits, long long ld, const void* bias, int tokens, int experts, int k, int softmax_all,
               int* ids, float* weights, cudaStream_t s) {
  if (tokens <= 0) return;
  if (experts > 256 || k > 8) throw std::runtime_error("moe_route: at most 256 experts and top-8");
  moe_route_kernel<<<(tokens + 3) / 4, 128, 0, s>>>((const __nv_bfloat16*)logits, ld, (const __nv_bfloat16*)bias,
                                                     tokens, experts, k, softmax_all, ids, weights);
  cuda_check(cudaGetLastError(), "moe_route_kernel");
}

// Single CTA. expert_lo/expert_hi select the experts this rank holds; entries routed elsewhere get
// row -1. Outputs: row_of[tokens*k] (permuted row of each (token, slot) or -1), token_of[rows_cap]
// (token of each permuted row, -1 = padding), tile_expert / tile_row0 / num_tiles, total_rows.
// Placement is deterministic: entries of an expert keep their (token, slot) order. Every warp owns a run of
// consecutive entries: it counts them per expert, a prefix over the warps gives each its first position,
// and on the second walk the lanes that drew the same expert rank themselves with a match mask. The warps
// never wait for one another inside a walk.
__global__ void __launch_bounds__(1024) moe_align_kernel(const int* __restrict__ ids, int entries, int expert_lo, int expert_hi, int bn, int k,
                                                         int* __restrict__ row_of, int* __restrict__ token_of,
                                                         int rows_cap, int* __restrict__ tile_expert,
                                                         int* __restrict__ tile_row0, int* __restrict__ num_tiles,
                                                         int max_tiles, const float* __restrict__ weights,
                                                         float* __restrict__ row_weight) {
  __shared__ int off[512], first_tile[512], cnt[512];
  extern __shared__ int fill[];               // [warp][local expert]: counts, then next positions
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int local = expert_hi - expert_lo;
  for (int i = threadIdx.x; i < warps * local; i += blockDim.x) fill[i] = 0;
  for (int i = threadIdx.x; i < rows_cap; i += blockDim.x) token_of[i] = -1;
  __syncthreads();
  int* mine = fill + warp * local;
  const int run = ((entries + warps - 1) / warps + 31) / 32 * 32, lo = warp * run, hi = min(lo + run, entries);
  for (int base = lo; base < hi; base += 32) {
    const int i = base + lane, e = i < hi ? ids[i] - expert_lo : -1;
    if (e >= 0 && e < local) atomicAdd(&mine[e], 1);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < local; e += blockDim.x) {
    int sum = 0;
    for (int w = 0; w < warps; ++w) {
      const int c = fill[w * local + e];
      fill[w * local + e] = sum;
      sum += c;
    }
    cnt[e] = (sum + bn - 1) / bn;             // tiles of the expert
  }
  __syncthreads();
  if (warp == 0) {                            // prefix of the tiles
    int done = 0;
    for (int base = 0; base < local; base += 32) {
      const int e = base + lane, c = e < local ? cnt[e] : 0;
      int p = c;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int q = __shfl_up_sync(0xffffffffu, p, o);
        if (lane >= o) p += q;
      }
      if (e < local) first_tile[e] = done + p - c, off[e] = (done + p - c) * bn;
      done += __shfl_sync(0xffffffffu, p, 31);
    }
    if (lane == 0) {
      num_tiles[0] = min(done, max_tiles);
      num_tiles[1] = done * bn;               // total permuted rows (incl. padding)
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < local; e += blockDim.x)
    for (int t = 0; t < cnt[e] && first_tile[e] + t < max_tiles; ++t) {
      tile_expert[first_tile[e] + t] = e;
      tile_row0[first_tile[e] + t] = off[e] + t * bn;
    }
  for (int base = lo; base < hi; base += 32) {
    const int i = base + lane, e = i < hi ? ids[i] - expert_lo : -1;
    const bool valid = e >= 0 && e < local;
    const unsigned same = __match_any_sync(0xffffffffu, valid ? e : -1 - lane);      // other lanes with this expert
    int pos = -1;
    if (valid) pos = off[e] + mine[e] + __popc(same & ((1u << lane) - 1u));
    __syncwarp();
    if (valid && lane == __ffs(same) - 1) mine[e] += __popc(same);
    __syncwarp();
    if (i < hi) row_of[i] = pos;
    if (valid && pos < rows_cap) {
      token_of[pos] = i / k;
      if (row_weight) row_weight[pos] = weights[i];
    }
  }
}

void moe_align(const int* ids, int tokens, int k, int expert_lo, int expert_hi, int bn, int* row_of,
               int* token_of, int rows_cap, int* tile_expert, int* tile_row0, int* num_tiles, int max_tiles,
               cudaStream_t s, const float* weights, float* row_weight) {
  if (expert_hi - expert_lo > 512) throw std::runtime_error("moe_align: at most 512 local experts");
  const size_t smem = (size_t)32 * std::max(expert_hi - expert_lo, 1) * sizeof(int);      // 64 KiB at most
  static bool configured[kMaxDevices] = {};
  if (first_call_on_device(configured))
    cuda_check(cudaFuncSetAttribute(moe_align_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024), "moe_align smem");
  moe_align_kernel<<<1, 1024, smem, s>>>(ids, tokens * k, expert_lo, expert_hi, bn, k, row_of, token_of, rows_cap, tile_expert, tile_row0, num_tiles,
                                         max_tiles, weights, row_weight);
  cuda_check(cudaGetLastError(), "moe_align_kernel");
}

// four values of a row as fp32
__device__ __forceinline__ float4 row4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 row4(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void put4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// row_weight (optional): routers that weigh an expert's input
template <typename T>
__global__ void moe_gather_kernel(const T* __restrict__ x, long long ldx, const int* __restrict__ token_of, const float* __restrict__ row_weight,
                                  T* __restrict__ xp, int hidden) {
  constexpr int V = 16 / sizeof(T);
  const int row = blockIdx.x;
  const int t = token_of[row];
  uint4* dst = reinterpret_cast<uint4*>(xp + (size_t)row * hidden);
  if (t < 0) {
    for (int i = threadIdx.x; i < hidden / V; i += blockDim.x) dst[i] = make_uint4(0, 0, 0, 0);
    return;
  }
  const T* src = x + (size_t)t * ldx;
  if (row_weight != nullptr) {
    const float w = row_weight[row];
    for (int i = threadIdx.x; i < hidden / 4; i += blockDim.x) {
      const float4 v = row4(src + 4 * i);
      put4(xp + (size_t)row * hidden + 4 * i, make_float4(v.x * w, v.y * w, v.z * w, v.w * w));
    }
    return;
  }
  for (int i = threadIdx.x; i < hidden / V; i += blockDim.x) dst[i] = reinterpret_cast<const uint4*>(src)[i];
}

void moe_gather(const void* x, long long ldx, const int* token_of, void* xp, int rows_cap, int hidden, cudaStream_t s, const float* row_weight, int f32) {
  if (rows_cap <= 0) return;
  if (f32) moe_gather_kernel<float><<<rows_cap, 128, 0, s>>>((const float*)x, ldx, token_of, row_weight, (float*)xp, hidden);
  else moe_gather_kernel<__nv_bfloat16><<<rows_cap, 128, 0, s>>>((const __nv_bfloat16*)x, ldx, token_of, row_weight, (__nv_bfloat16*)xp, hidden);
  cuda_check(cudaGetLastError(), "moe_gather_kernel");
}

// weights (optional; none: the rows are summed as they are), add (optional): rows added to the result, each times add_gate (optional)
template <typename T>
__global__ void moe_combine_kernel(const T* __restrict__ y, long long ldy, const int* __restrict__ row_of, const float* __restrict__ weights, int k,
                                   const T* __restrict__ add, long long ld_add, const float* __restrict__ add_gate, T* __restrict__ out, long long ldo,
                                   int hidden) {
  const int t = blockIdx.x;
  const float ga = add_gate != nullptr ? add_gate[t] : 1.f;
  for (int i = threadIdx.x; i < hidden / 4; i += blockDim.x) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int j = 0; j < k; ++j) {
      const int row = row_of[(size_t)t * k + j];
      if (row < 0) continue;                                  // expert lives on another rank
      const float w = weights != nullptr ? weights[(size_t)t * k + j] : 1.f;
      const float4 v = row4(y + (size_t)row * ldy + 4 * i);
      acc.x += w * v.x, acc.y += w * v.y, acc.z += w * v.z, acc.w += w * v.w;
    }
    if (add != nullptr) {
      const float4 v = row4(add + (size_t)t * ld_add + 4 * i);
      acc.x = fmaf(ga, v.x, acc.x), acc.y = fmaf(ga, v.y, acc.y), acc.z = fmaf(ga, v.z, acc.z), acc.w = fmaf(ga, v.w, acc.w);
    }
    put4(out + (size_t)t * ldo + 4 * i, acc);
  }
}

void moe_combine(const void* y, long long ldy, const int* row_of, const float* weights, int tokens, int k, void* out,
                 long long ldo, int hidden, cudaStream_t s, const void* add, long long ld_add, int f32, const float* add_gate) {
  if (tokens <= 0) return;
  if (f32)
    moe_combine_kernel<float><<<tokens, 128, 0, s>>>((const float*)y, ldy, row_of, weights, k, (const float*)add, ld_add, add_gate, (float*)out, ldo,
                                                      hidden);
  else
    moe_combine_kernel<__nv_bfloat16><<<tokens, 128, 0, s>>>((const __nv_bfloat16*)y, ldy, row_of, weights, k, (const __nv_bfloat16*)add, ld_add,
                                                              add_gate, (__nv_bfloat16*)out, ldo, hidden);
  cuda_check(cudaGetLastError(), "moe_combine_kernel");
}

}  // namespace fllm
