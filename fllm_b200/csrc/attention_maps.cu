// Attention of one or two maps over shared values, with key and value rows of widths of their own and a sliding window:
//   a_m = softmax_j(scale q_m . k_m,j) v_j over the keys j with 0 <= i - j < window (window 0: all up to i)
//   one map: out = a_1;  two maps (differential attention): out = rms(a_1 - lam a_2) * out_scale over the head's values
// With a sink the denominator of one map also holds exp(sink of the head). With a distance bias (one map) r1 ln(1 + r2 (i - j)) of the
// head is taken off a score. "Spread" attention weighs the values of every key/value head with every head's weights (one value row
// per token holds them all) and leaves fp32 partial sums; talk_mix adds them up with a matrix over the heads, which is the same as
// mixing the heads' weights in front of the values, and gates the heads.
// Rows are padded with zeros to wk and wv (64, 128, or a multiple of 16 above). Pools: keys [block][kv head][map][token][wk],
// values [block][kv head][token][wv]; queries [token][head][map][wk]. Query rows of a sequence are numbered token * group + head
// within one kv head.
//
//   maps_prepare_kernel  projection -> normalised, rotated queries; normalised, rotated keys and values into the pools
//   maps_prefill_kernel  tcgen05 with accumulators in tensor memory. A CTA runs two streams of 128 query rows with a score and an
//                        output accumulator each: the two maps of the same rows, or (one map) two neighbouring row tiles. The
//                        softmax of one stream runs under the products of the other, and both read the same V tile.
//   maps_decode_kernel   mma.sync, 16 query rows per CTA (two maps: 8 rows of each), each warp streaming its own 16-token pages
//                        through a private cp.async ring; split over key slices.
//   maps_simple_kernel   CUDA cores, any width, bf16 and fp32.
// (Spread attention on the tensor cores and the mixing of its heads: attention_talk.cu.)
//
// Weights are fp32; for the tensor-core product with the values a weight travels as the sum of two bf16 values (16 significant
// bits). The maps are combined in fp32 before anything is rounded. Nothing in front of a window's first page is read.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>
#include <stdexcept>
#include <unordered_map>

#include "attention_util.cuh"
#include "fllm_ops.h"
#include "ptx.cuh"
#include "tma_host.h"

namespace fllm {
namespace {
constexpr int kDecodeRows = 64;           // sequences with at most this many query rows per kv head run in the decode kernel

// ------------------------------------------------------------------------------------------ queries and cache rows
// One CTA per (token, share of its maps and value heads), a warp per map at a time.
constexpr int kMaxTaps = 8;
template <typename T, bool CONV>
__global__ void __launch_bounds__(128) maps_prepare_kernel(const MapsPrepareParams p) {
  extern __shared__ float sm[];
  float2* turn = reinterpret_cast<float2*>(sm);                   // [rot / 2] cosine, sine
  float* buf = sm + p.rot + (threadIdx.x >> 5) * p.dim;           // [4][dim]
  __shared__ float2 red[4];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int pos = p.positions[t], slot = p.slots[t], half = p.rot / 2;
  const T* xr = static_cast<const T*>(p.x) + (long long)t * p.ldx;
  const float* part = p.partials ? p.partials + (size_t)t * p.width : nullptr;
  const T* bias = static_cast<const T*>(p.bias);
  // short convolution of steps in which every sequence has one token: the taps before it come from the sequence's state row,
  // which moves on by one token where `write` is set
  T* window = CONV ? static_cast<T*>(p.conv_state) + (long long)p.seq_state[t] * (p.taps - 1) * p.conv_width : nullptr;
  const bool fresh = pos == 0;
  auto conv1 = [&](int c, float u, bool write) {
    const float* w = p.conv_w + (long long)c * p.taps;
    float v = w[p.taps - 1] * u, next = u;
    for (int j = p.taps - 2; j >= 0; --j) {
      T* at = window + (long long)j * p.conv_width + c;
      const float old = fresh ? 0.f : to_f32(*at);
      v = fmaf(w[j], old, v);
      if (write) *at = from_f32<T>(next);
      next = old;
    }
    return v;
  };
  auto conv4 = [&](int c, const float4& u, bool write) {          // four columns from a multiple of 4 on: all loads in flight at once
    using Raw = typename Four<T>::type;
    Raw old[kMaxTaps - 1];
    float4 w[kMaxTaps];
#pragma unroll
    for (int j = 0; j < kMaxTaps - 1; ++j)
      if (j < p.taps - 1) old[j] = fresh ? Raw{} : *reinterpret_cast<const Raw*>(window + (long long)j * p.conv_width + c);
    const float* wc = p.conv_w + (long long)c * p.taps;
    if (p.taps == 4) {                                            // 4 x 4, a row per column
      const float4 r0 = *reinterpret_cast<const float4*>(wc), r1 = *reinterpret_cast<const float4*>(wc + 4), r2 = *reinterpret_cast<const float4*>(wc + 8),
                   r3 = *reinterpret_cast<const float4*>(wc + 12);
      w[0] = make_float4(r0.x, r1.x, r2.x, r3.x), w[1] = make_float4(r0.y, r1.y, r2.y, r3.y);
      w[2] = make_float4(r0.z, r1.z, r2.z, r3.z), w[3] = make_float4(r0.w, r1.w, r2.w, r3.w);
    } else {
#pragma unroll
      for (int j = 0; j < kMaxTaps; ++j)
        if (j < p.taps) w[j] = make_float4(wc[j], wc[p.taps + j], wc[2 * p.taps + j], wc[3 * p.taps + j]);
    }
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j) {
      if (j < p.taps - 1) {
        const T* e = reinterpret_cast<const T*>(&old[min(j, kMaxTaps - 2)]);
        v.x = fmaf(w[j].x, to_f32(e[0]), v.x), v.y = fmaf(w[j].y, to_f32(e[1]), v.y);
        v.z = fmaf(w[j].z, to_f32(e[2]), v.z), v.w = fmaf(w[j].w, to_f32(e[3]), v.w);
        if (write && j > 0) *reinterpret_cast<Raw*>(window + (long long)(j - 1) * p.conv_width + c) = old[min(j, kMaxTaps - 2)];
      } else if (j == p.taps - 1) {
        v.x = fmaf(w[j].x, u.x, v.x), v.y = fmaf(w[j].y, u.y, v.y), v.z = fmaf(w[j].z, u.z, v.z), v.w = fmaf(w[j].w, u.w, v.w);
      }
    }
    if (write) {
      const float f[4] = {u.x, u.y, u.z, u.w};
      Raw raw;
      T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
      for (int i = 0; i < 4; ++i) e[i] = from_f32<T>(f[i]);
      *reinterpret_cast<Raw*>(window + (long long)(p.taps - 2) * p.conv_width + c) = raw;
    }
    return v;
  };
  auto load1 = [&](int c) {
    float v = bias ? to_f32(bias[c]) : 0.f;
    if (!part) return v + to_f32(xr[c]);
    for (int s = 0; s < p.splits; ++s) v += __ldcg(part + s * p.plane + c);
    return v;
  };
  // columns base + c .. c + 3 of a segment of n values, zeros behind it
  auto raw4 = [&](int base, int c, int n) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.vec) {                                                  // n is a multiple of 4
      if (c >= n) return v;
      if (part) {
        for (int s = 0; s < p.splits; ++s) {
          const float4 q = __ldcg(reinterpret_cast<const float4*>(part + s * p.plane + base + c));
          v.x += q.x, v.y += q.y, v.z += q.z, v.w += q.w;
        }
      }
      auto plus = [&](const T* src) {
        const typename Four<T>::type raw = *reinterpret_cast<const typename Four<T>::type*>(src + base + c);
        const T* e = reinterpret_cast<const T*>(&raw);
        v.x += to_f32(e[0]), v.y += to_f32(e[1]), v.z += to_f32(e[2]), v.w += to_f32(e[3]);
      };
      if (!part) plus(xr);
      if (bias) plus(bias);
      return v;
    }
    float* f = &v.x;
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (c + e < n) f[e] = load1(base + c + e);
    return v;
  };
  // behind the convolution, if any: with `write` the state row moves on, so every column is loaded once with it
  auto load4 = [&](int base, int c, int n, bool write) {
    float4 v = raw4(base, c, n);
    if (CONV && p.vec) {
      if (c < n) v = conv4(base + c, v, write);
    } else if (CONV) {
      float* f = &v.x;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < n) f[e] = conv1(base + c + e, f[e], write);
    }
    return v;
  };
  auto store4 = [](T* dst, const float (&v)[4]) {
    typename Four<T>::type raw;
    T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) e[i] = from_f32<T>(v[i]);
    *reinterpret_cast<typename Four<T>::type*>(dst) = raw;
  };
  auto sq = [](const float4& v) { return fmaf(v.x, v.x, v.y * v.y) + fmaf(v.z, v.z, v.w * v.w); };

  for (int i = threadIdx.x; i < half; i += 128) {
    float s, c;
    sincosf((float)pos * p.inv_freq[i], &s, &c);
    turn[i] = make_float2(c * p.rope_factor, s * p.rope_factor);
  }
  float2 all = make_float2(0.f, 0.f);                             // full: 1 / rms of all query maps and of all key maps
  if (p.full) {
    float2 ss = make_float2(0.f, 0.f);
    for (int c = 4 * threadIdx.x; c < p.q_heads * p.dim; c += 512) ss.x += sq(load4(p.q_offset, c, p.q_heads * p.dim, false));
    for (int c = 4 * threadIdx.x; c < p.k_heads * p.dim; c += 512) ss.y += sq(load4(p.k_offset, c, p.k_heads * p.dim, false));
    ss = make_float2(warp_sum(ss.x), warp_sum(ss.y));
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    for (int w = 0; w < 4; ++w) all.x += red[w].x, all.y += red[w].y;
    all.x = 1.f / sqrtf(all.x / (float)(p.q_heads * p.dim) + p.eps), all.y = 1.f / sqrtf(all.y / (float)(p.k_heads * p.dim) + p.eps);
  }
  __syncthreads();
  if (p.lanes > 0) {
    // maps of up to 64 or 128 values: 16 or 32 lanes with four values each, so that a warp has one or two maps at a time and a
    // rotation partner is a shuffle away, or in the same lane
    const int maps = p.q_heads + (slot >= 0 ? p.k_heads : 0), per = 32 / p.lanes, sub = lane / p.lanes, li = lane % p.lanes, c = 4 * li;
    const bool low = c < half, turns = c < p.rot;
    const int mate = turns && !p.pairs ? lane + (low ? half / 4 : -half / 4) : lane;
    float2 cs[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) cs[e] = turns ? turn[p.pairs ? (c + e) / 2 : (low ? c : c - half) + e] : make_float2(1.f, 0.f);
    for (int i0 = (blockIdx.y * 4 + warp) * per; i0 < maps; i0 += 4 * per * gridDim.y) {
      const int item = min(i0 + sub, maps - 1);                   // (lanes past the end repeat the last map)
      const bool is_q = item < p.q_heads;
      const int h = is_q ? item : item - p.q_heads;
      const float4 f = load4((is_q ? p.q_offset : p.k_offset) + h * p.dim, c, p.dim, i0 + sub < maps);
      float ss = sq(f);
      for (int o = p.lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float inv = p.eps < 0.f ? 1.f : (p.full ? (is_q ? all.x : all.y) : 1.f / sqrtf(ss / (float)p.dim + p.eps));
      float v[4] = {f.x * inv, f.y * inv, f.z * inv, f.w * inv};
      if (p.q_norm != nullptr && c < p.dim) {
        const T* w = static_cast<const T*>(is_q ? p.q_norm : p.k_norm) + (p.full ? h * p.dim : 0) + c;
        const typename Four<T>::type raw = *reinterpret_cast<const typename Four<T>::type*>(w);
        const T* wv = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] *= to_f32(wv[e]);
      }
      if (p.pairs) {
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const float a = v[e], b = v[e + 1];
          v[e] = a * cs[e].x - b * cs[e].y, v[e + 1] = b * cs[e].x + a * cs[e].y;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float m = __shfl_sync(0xffffffffu, v[e], mate);
          v[e] = low ? v[e] * cs[e].x - m * cs[e].y : v[e] * cs[e].x + m * cs[e].y;
        }
      }
      T* dst = is_q ? static_cast<T*>(p.q_out) + ((long long)t * p.q_heads + h) * p.wk
                    : static_cast<T*>(p.k_cache) + (((long long)(slot / p.block_size) * p.k_heads + h) * p.block_size + slot % p.block_size) * p.wk;
      if (i0 + sub < maps) store4(dst + c, v);
    }
  }
  const int items = p.q_heads + (slot >= 0 ? p.k_heads + p.v_heads : 0);
  const long long block = slot >= 0 ? slot / p.block_size : 0;
  const int at = slot >= 0 ? slot % p.block_size : 0;
  for (int item = (p.lanes > 0 ? p.q_heads + p.k_heads : 0) + blockIdx.y * 4 + warp; item < items; item += 4 * gridDim.y) {
    float v[4];
    if (item >= p.q_heads + p.k_heads) {                          // values go to the pool as they are
      const int g = item - p.q_heads - p.k_heads;
      T* dst = static_cast<T*>(p.v_cache) + ((block * p.v_heads + g) * p.block_size + at) * p.wv;
      for (int c = 4 * lane; c < p.wv; c += 128) {
        const float4 f = load4(p.v_offset + g * p.v_dim, c, p.v_dim, true);
        v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
        store4(dst + c, v);
      }
      continue;
    }
    const bool is_q = item < p.q_heads;
    const int h = is_q ? item : item - p.q_heads;
    const int base = (is_q ? p.q_offset : p.k_offset) + h * p.dim;
    const T* w = p.q_norm ? static_cast<const T*>(is_q ? p.q_norm : p.k_norm) + (p.full ? h * p.dim : 0) : nullptr;
    T* dst = is_q ? static_cast<T*>(p.q_out) + ((long long)t * p.q_heads + h) * p.wk
                  : static_cast<T*>(p.k_cache) + ((block * p.k_heads + h) * p.block_size + at) * p.wk;
    float ss = 0.f;
    for (int c = 4 * lane; c < p.dim; c += 128) {
      const float4 f = load4(base, c, p.dim, true);
      ss += sq(f);
      buf[c] = f.x;
      if (c + 1 < p.dim) buf[c + 1] = f.y;
      if (c + 2 < p.dim) buf[c + 2] = f.z;
      if (c + 3 < p.dim) buf[c + 3] = f.w;
    }
    const float own = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps), inv = p.eps < 0.f ? 1.f : (p.full ? (is_q ? all.x : all.y) : own);
    __syncwarp();
    for (int c = 4 * lane; c < p.wk; c += 128) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = c + e;
        v[e] = 0.f;
        if (i >= p.dim) continue;
        const float n = buf[i] * inv * (w ? to_f32(w[i]) : 1.f);
        v[e] = n;
        if (i < p.rot) {
          const bool low = p.pairs ? i % 2 == 0 : i < half;
          const int step = p.pairs ? 1 : half, j = low ? i + step : i - step;
          const float2 cs = turn[p.pairs ? i / 2 : min(i, j)];
          const float m = buf[j] * inv * (w ? to_f32(w[j]) : 1.f);
          v[e] = low ? n * cs.x - m * cs.y : n * cs.x + m * cs.y;
        }
      }
      store4(dst + c, v);
    }
    __syncwarp();
  }
  // further columns of the projection, as fp32
  if (blockIdx.y == 0)
    for (int i = threadIdx.x; i < p.extra; i += 128) p.extra_out[(long long)t * p.extra + i] = load1(p.extra_offset + i);
}

// ------------------------------------------------------------------------------------------ CUDA-core attention
// One CTA per (head, token) and, for spread attention, piece of E * 32 value columns; its warps take every NW-th key with an online
// softmax each and are merged through shared memory.
template <typename T, int E, int M, int NW>
__global__ void __launch_bounds__(NW * 32) maps_simple_kernel(const MapsAttnParams p) {
  extern __shared__ float sm[];
  const int col0 = blockIdx.z * E * 32, v_dim = min(p.v_dim - col0, E * 32);
  float* sq = sm;                              // [M][dim] query rows
  float* sacc = sq + M * p.dim;                // [M][NW][v_dim]
  float* sml = sacc + M * NW * v_dim;          // [M][NW][2] maximum and sum
  __shared__ float red[NW];
  const int h = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (p.H / p.G);
  const float r1 = p.r1 ? p.r1[h] : 0.f, r2 = p.r1 ? p.r2[h] : 0.f;
  const T* q = static_cast<const T*>(p.q) + ((long long)t * p.H + h) * M * p.wk;
  const T* kc = static_cast<const T*>(p.k_cache);
  const T* vc = static_cast<const T*>(p.v_cache);
  for (int i = threadIdx.x; i < M * p.dim; i += NW * 32) sq[i] = to_f32(q[(i / p.dim) * p.wk + i % p.dim]);
  __syncthreads();
  const int kv_len = p.positions[t] + 1, first = p.window > 0 ? max(0, kv_len - p.window) : 0;
  const int* table = p.block_tables + (size_t)p.row_seq[t] * p.max_blocks;
  float m[M], l[M], acc[M][E];
#pragma unroll
  for (int a = 0; a < M; ++a) {
    m[a] = -INFINITY, l[a] = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) acc[a][e] = 0.f;
  }
  for (int j = first + warp; j < kv_len; j += NW) {
    const size_t block = (size_t)table[j / p.block_size] * p.G + g;
    const int at = j % p.block_size;
    const size_t vblock = p.spread ? (size_t)table[j / p.block_size] : block;
    const T* vr = vc + (vblock * p.block_size + at) * p.wv + col0;
    float v[E];
#pragma unroll
    for (int e = 0; e < E; ++e) v[e] = lane + 32 * e < v_dim ? to_f32(vr[lane + 32 * e]) : 0.f;
#pragma unroll
    for (int a = 0; a < M; ++a) {
      const T* kr = kc + ((block * M + a) * p.block_size + at) * p.wk;
      float s = 0.f;
#pragma unroll 4
      for (int c = lane; c < p.dim; c += 32) s = fmaf(to_f32(kr[c]), sq[a * p.dim + c], s);
      s = warp_sum(s) * p.scale;
      if (p.r1) s -= r1 * log1pf(r2 * (float)(kv_len - 1 - j));
      const float mn = fmaxf(m[a], s), corr = expf(m[a] - mn), pr = expf(s - mn);
      l[a] = l[a] * corr + pr;
#pragma unroll
      for (int e = 0; e < E; ++e) acc[a][e] = fmaf(acc[a][e], corr, pr * v[e]);
      m[a] = mn;
    }
  }
#pragma unroll
  for (int a = 0; a < M; ++a) {
#pragma unroll
    for (int e = 0; e < E; ++e)
      if (lane + 32 * e < v_dim) sacc[(a * NW + warp) * v_dim + lane + 32 * e] = acc[a][e];
    if (lane == 0) sml[2 * (a * NW + warp)] = m[a], sml[2 * (a * NW + warp) + 1] = l[a];
  }
  __syncthreads();
  float c[M][NW], tot[M], mm;
#pragma unroll
  for (int a = 0; a < M; ++a) {
    mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < NW; ++w) mm = fmaxf(mm, sml[2 * (a * NW + w)]);
    tot[a] = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) {
      const float mw = sml[2 * (a * NW + w)];
      c[a][w] = mw == -INFINITY ? 0.f : expf(mw - mm);
      tot[a] = fmaf(sml[2 * (a * NW + w) + 1], c[a][w], tot[a]);
    }
  }
  if (p.spread) {                              // partial sums of one key slice
    const size_t row = (size_t)t * p.H + h;
    for (int i = threadIdx.x; i < v_dim; i += NW * 32) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < NW; ++w) v = fmaf(sacc[w * v_dim + i], c[0][w], v);
      p.part_o[row * p.wv + col0 + i] = v;
    }
    if (threadIdx.x == 0 && col0 == 0) p.part_ml[2 * row] = mm, p.part_ml[2 * row + 1] = tot[0];
    return;
  }
  if (M == 1 && p.sink) tot[0] += expf(p.sink[h] - mm);
  auto value = [&](int i) {
    float o = 0.f;
#pragma unroll
    for (int a = 0; a < M; ++a) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < NW; ++w) v = fmaf(sacc[(a * NW + w) * v_dim + i], c[a][w], v);
      o = a == 0 ? v / tot[0] : o - p.lam * (v / tot[a]);
    }
    return o;
  };
  float f = 1.f;
  if (M == 2) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.v_dim; i += NW * 32) {
      const float o = value(i);
      ss = fmaf(o, o, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) ss += red[w];
    f = p.out_scale / sqrtf(ss / (float)p.v_dim + p.eps);
  }
  T* out = static_cast<T*>(p.out) + (long long)t * p.ldo + h * p.v_dim;
  for (int i = threadIdx.x; i < p.v_dim; i += NW * 32) out[i] = from_f32<T>(value(i) * f);
}

// ------------------------------------------------------------------------------------------ shared by the tensor-core kernels
struct Maps {
  const bf16 *q, *kc, *vc;
  const int* block_tables;
  int max_blocks;
  const int *q_starts, *positions;
  bf16* out;
  long long ldo;
  int H, G, group, v_dim, block_size, vec;   // vec: output rows can be stored in 16-byte pieces
  int window;
  float scale_log2, lam, out_scale, eps;
  float *ws_o, *ws_ml;                       // partial results of key slices: [T][H][maps][splits][DV], [T][H][maps][splits][2]
  int splits;
  int* status;
  const float* sink;                         // optional [H], natural units
};

// first pool row of the kPage tokens from `token` on, in a pool of `heads` rows per token
__device__ __forceinline__ int page_row(const Maps& p, const int* table, int token, int heads, int head) {
  return (table[token / p.block_size] * heads + head) * p.block_size + token % p.block_size;
}
__device__ __forceinline__ int first_key(const Maps& p, int lim) { return p.window > 0 ? max(0, lim - p.window) : 0; }

// what a head's sink adds to a sum of weights whose reference is m (log2 units)
__device__ __forceinline__ float sink_weight(const Maps& p, int head, float m) { return p.sink ? ex2(p.sink[head] * kLog2e - m) : 0.f; }

// one warp, lane holding the values lane + 32 e of every map's weighted sum, the sums of its weights and their reference
template <int M, int E>
__device__ __forceinline__ void finish_row(const Maps& p, long long tok, int head, const float (&a)[M][E], const float (&l)[M], float m, int lane) {
  float y[E], ss = 0.f, f = 1.f;
  const float l0 = M == 1 ? l[0] + sink_weight(p, head, m) : l[0], i0 = l0 > 0.f ? 1.f / l0 : 0.f, i1 = M == 2 && l[M - 1] > 0.f ? p.lam / l[M - 1] : 0.f;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    y[e] = a[0][e] * i0;
    if (M == 2) y[e] -= a[M - 1][e] * i1;
    ss = fmaf(y[e], y[e], ss);                             // the padding is zero
  }
  if (M == 2) f = p.out_scale / sqrtf(warp_sum(ss) / (float)p.v_dim + p.eps);
  bf16* dst = p.out + tok * p.ldo + (long long)head * p.v_dim;
#pragma unroll
  for (int e = 0; e < E; ++e)
    if (lane + 32 * e < p.v_dim) dst[lane + 32 * e] = __float2bfloat16(y[e] * f);
}

// ------------------------------------------------------------------------------------------ decode
template <int DK, int DV, int M>
struct DecodeTile {
  static constexpr int kKey = kPage * DK * 2, kStage = M * kKey + kPage * DV * 2;      // key rows of every map, then the values
  static constexpr int kStages = kStage <= 4096 ? 6 : (kStage <= 6144 ? 4 : (kStage <= 8192 ? 3 : 2));
  static constexpr int kQ = 16 * DK * 2, kRing = 4 * kStages * kStage;
  static constexpr int kMerge = 4 * 16 * DV * 4 + 4 * 16 * 2 * 4;
  static constexpr int kTotal = kQ + (kRing > kMerge ? kRing : kMerge) + 128;
  static constexpr int kRowsOf = 16 / M;                   // query rows of a tile: row r of map m is tile row m * kRowsOf + r
};

template <int DK, int DV, int M>
__global__ void __launch_bounds__(128, 2) maps_decode_kernel(const Maps p, int row_tiles, int max_rows) {
  using L = DecodeTile<DK, DV, M>;
  constexpr int R = L::kRowsOf;
  extern __shared__ __align__(128) uint8_t smem[];
  bf16* qtile = reinterpret_cast<bf16*>(smem);
  uint8_t* ring = smem + L::kQ;
  const int kvh = blockIdx.x / row_tiles, row0 = (blockIdx.x % row_tiles) * R, seq = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0;
  const int all_rows = qn * p.group;
  if (qn <= 0 || all_rows > max_rows || row0 >= all_rows) return;
  const int n_rows = min(R, all_rows - row0);
  const int kv_len = p.positions[q0 + qn - 1] + 1, first_pos = kv_len - qn;
  const int hi_tok = first_pos + (row0 + n_rows - 1) / p.group + 1;
  const int page0 = first_key(p, first_pos + row0 / p.group + 1) / kPage, pages = (hi_tok + kPage - 1) / kPage - page0;
  const int per = (pages + p.splits - 1) / p.splits;
  const int pg0 = page0 + split * per, pg1 = page0 + min((split + 1) * per, pages);

  for (int i = threadIdx.x; i < 16 * (DK / 8); i += 128) {
    const int r = i / (DK / 8), c = i - r * (DK / 8), sub = r % R;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (sub < n_rows) {
      const long long head = (long long)(q0 + (row0 + sub) / p.group) * p.H + kvh * p.group + (row0 + sub) % p.group;
      v = *reinterpret_cast<const uint4*>(p.q + (head * M + r / R) * DK + c * 8);
    }
    *reinterpret_cast<uint4*>(tile_ptr<DK>(qtile, r, c)) = v;
  }
  __syncthreads();
  uint32_t qf[DK / 16][4];
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk) ldsm_x4(qf[kk], tile_ptr<DK>(qtile, lane & 15, 2 * kk + (lane >> 4)));

  const int g = lane >> 2, t4 = lane & 3;
  int lim[2], beg[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int sub = (g + 8 * i) % R;
    lim[i] = sub < n_rows ? first_pos + (row0 + sub) / p.group + 1 : 0;
    beg[i] = first_key(p, lim[i]);
  }
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};

  uint8_t* mine = ring + (size_t)warp * L::kStages * L::kStage;
  const int* table = p.block_tables + (size_t)seq * p.max_blocks;
  auto issue = [&](int it) {
    const int pg = pg0 + warp + 4 * it;
    if (pg < pg1) {
      uint8_t* st = mine + (size_t)(it % L::kStages) * L::kStage;
#pragma unroll
      for (int a = 0; a < M; ++a) {
        const bf16* src = p.kc + (long long)page_row(p, table, pg * kPage, p.G * M, kvh * M + a) * DK;
#pragma unroll
        for (int i = lane; i < kPage * (DK / 8); i += 32) {
          const int r = i / (DK / 8), c = i - r * (DK / 8);
          cp_async16(tile_ptr<DK>(reinterpret_cast<bf16*>(st + a * L::kKey), r, c), src + (size_t)r * DK + c * 8);
        }
      }
      const bf16* src = p.vc + (long long)page_row(p, table, pg * kPage, p.G, kvh) * DV;
#pragma unroll
      for (int i = lane; i < kPage * (DV / 8); i += 32) {
        const int r = i / (DV / 8), c = i - r * (DV / 8);
        cp_async16(tile_ptr<DV>(reinterpret_cast<bf16*>(st + M * L::kKey), r, c), src + (size_t)r * DV + c * 8);
      }
    }
    cp_async_commit();
  };
  const int my_pages = pg1 > pg0 + warp ? (pg1 - pg0 - warp + 3) / 4 : 0;
#pragma unroll
  for (int s = 0; s < L::kStages - 1; ++s) issue(s);
  for (int it = 0; it < my_pages; ++it) {
    issue(it + L::kStages - 1);
    cp_async_wait<L::kStages - 1>();
    __syncwarp();
    uint8_t* st = mine + (size_t)(it % L::kStages) * L::kStage;
    bf16* vs = reinterpret_cast<bf16*>(st + M * L::kKey);
    const int tok_base = (pg0 + warp + 4 * it) * kPage, j4 = lane >> 3;
    float s[M][2][4];
#pragma unroll
    for (int a = 0; a < M; ++a) {
#pragma unroll
      for (int i = 0; i < 2; ++i) s[a][i][0] = s[a][i][1] = s[a][i][2] = s[a][i][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t b[4];
        ldsm_x4(b, tile_ptr<DK>(reinterpret_cast<bf16*>(st + a * L::kKey), (j4 >> 1) * 8 + (lane & 7), 2 * kk + (j4 & 1)));
        mma_bf16(s[a][0], qf[kk], b[0], b[1]);
        mma_bf16(s[a][1], qf[kk], b[2], b[3]);
      }
    }
    // ---- weights of two rows x four tokens (two maps: the upper eight rows of the tile are the second map's)
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = e >> 1, tok = tok_base + nb * 8 + 2 * t4 + (e & 1);
        const float v = s[M == 2 ? i : 0][nb][e] * p.scale_log2;
        s[0][nb][e] = tok >= beg[i] && tok < lim[i] ? v : -INFINITY;
        mx[i] = fmaxf(mx[i], s[0][nb][e]);
      }
    }
    float ref[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
      const float mn = fmaxf(m[i], mx[i]);
      ref[i] = mn == -INFINITY ? 0.f : mn;
      const float c = ex2(m[i] - ref[i]);
      l[i] *= c;
      m[i] = mn;
#pragma unroll
      for (int db = 0; db < DV / 8; ++db) o[db][2 * i] *= c, o[db][2 * i + 1] *= c;
    }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float p0 = ex2(s[0][nb][2 * i] - ref[i]), p1 = ex2(s[0][nb][2 * i + 1] - ref[i]);
        l[i] += p0 + p1;
        const uint32_t hi = pack_bf16x2(p0, p1);
        const float2 back = unpack_bf16x2(hi);
        ph[nb * 2 + i] = hi;
        pl[nb * 2 + i] = pack_bf16x2(p0 - back.x, p1 - back.y);
      }
#pragma unroll
    for (int db = 0; db < DV / 8; db += 2) {
      uint32_t b[4];
      ldsm_x4_t(b, tile_ptr<DV>(vs, (j4 & 1) * 8 + (lane & 7), db + (j4 >> 1)));
      mma_bf16(o[db], ph, b[0], b[1]);
      mma_bf16(o[db + 1], ph, b[2], b[3]);
      mma_bf16(o[db], pl, b[0], b[1]);
      mma_bf16(o[db + 1], pl, b[2], b[3]);
    }
    __syncwarp();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
  }
  __syncthreads();                                       // the rings are free: merge the four warps
  float* mo = reinterpret_cast<float*>(smem + L::kQ);    // [4][16][DV]
  float* mml = mo + 4 * 16 * DV;                         // [4][16][2]
#pragma unroll
  for (int db = 0; db < DV / 8; ++db) {
    *reinterpret_cast<float2*>(mo + ((size_t)warp * 16 + g) * DV + db * 8 + 2 * t4) = make_float2(o[db][0], o[db][1]);
    *reinterpret_cast<float2*>(mo + ((size_t)warp * 16 + g + 8) * DV + db * 8 + 2 * t4) = make_float2(o[db][2], o[db][3]);
  }
  if (t4 == 0) {
#pragma unroll
    for (int i = 0; i < 2; ++i) mml[(warp * 16 + g + 8 * i) * 2] = m[i], mml[(warp * 16 + g + 8 * i) * 2 + 1] = l[i];
  }
  __syncthreads();
  constexpr int E = DV / 32;
  for (int sub = warp; sub < n_rows; sub += 4) {
    const int head = kvh * p.group + (row0 + sub) % p.group;
    const long long tok = q0 + (row0 + sub) / p.group;
    float a[M][E], ls[M], ms[M];
#pragma unroll
    for (int k = 0; k < M; ++k) {
      const int r = k * R + sub;
      ms[k] = -INFINITY, ls[k] = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) ms[k] = fmaxf(ms[k], mml[(w * 16 + r) * 2]);
#pragma unroll
      for (int e = 0; e < E; ++e) a[k][e] = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float mw = mml[(w * 16 + r) * 2];
        const float c = mw == -INFINITY ? 0.f : ex2(mw - ms[k]);
        ls[k] = fmaf(mml[(w * 16 + r) * 2 + 1], c, ls[k]);
#pragma unroll
        for (int e = 0; e < E; ++e) a[k][e] = fmaf(mo[((size_t)w * 16 + r) * DV + lane + 32 * e], c, a[k][e]);
      }
    }
    if (p.splits == 1) {
      finish_row<M, E>(p, tok, head, a, ls, ms[0], lane);
      continue;
    }
#pragma unroll
    for (int k = 0; k < M; ++k) {
      const size_t base = ((tok * p.H + head) * M + k) * p.splits + split;
#pragma unroll
      for (int e = 0; e < E; ++e) p.ws_o[base * DV + lane + 32 * e] = a[k][e];
      if (lane == 0) p.ws_ml[base * 2] = ms[k], p.ws_ml[base * 2 + 1] = ls[k];
    }
  }
}

// one warp per (token, head)
template <int DV, int M>
__global__ void __launch_bounds__(128) maps_merge_kernel(const Maps p, int T) {
  constexpr int E = DV / 32;
  pdl_launch_dependents();
  pdl_wait();
  const int item = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= T * p.H) return;
  float a[M][E], l[M], mm;
#pragma unroll
  for (int k = 0; k < M; ++k) {
    const size_t base = ((size_t)item * M + k) * p.splits;
    mm = -INFINITY;
    l[k] = 0.f;
    for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, p.ws_ml[(base + s) * 2]);
#pragma unroll
    for (int e = 0; e < E; ++e) a[k][e] = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float ms = p.ws_ml[(base + s) * 2];
      if (ms == -INFINITY) continue;
      const float w = ex2(ms - mm);
      l[k] = fmaf(p.ws_ml[(base + s) * 2 + 1], w, l[k]);
#pragma unroll
      for (int e = 0; e < E; ++e) a[k][e] = fmaf(p.ws_o[(base + s) * DV + lane + 32 * e], w, a[k][e]);
    }
  }
  finish_row<M, E>(p, item / p.H, item % p.H, a, l, mm, lane);
}

// ------------------------------------------------------------------------------------------ prefill
// Warp 0 brings K and V tiles (eight pages of 16 rows by TMA, 128-byte swizzle), warp 1 issues the MMAs, warps 2 - 5 and 6 - 9 are
// the softmax of the two streams, one thread per query row. The weights of 32 tokens overwrite the 32 columns their scores came
// from: 16 columns of leading bf16 terms, 16 of remainders. Tensor memory: S / P of the streams 2 x 128 columns, O 2 x 128.
// Order of the products: S_0, S_1 of the first tile, then per tile O_0, next S_0, O_1, next S_1: while one stream waits for its
// weights the other's products run. Every wait is bounded.
constexpr int kThreads = 320;
template <int DK, int DV, int M>
struct PrefillTile {
  static constexpr int kQ = 2 * tile_bytes<DK>(), kK = M * tile_bytes<DK>(), kV = tile_bytes<DV>(), kTail = 256 + 2 * 128 * 4 * 2;
  static constexpr int kStages = kQ + 2 * (kK + kV) + kTail + 1024 <= 227 * 1024 ? 2 : 1;
  static constexpr int kUsed = kQ + kStages * (kK + kV) + kTail + 1024;
  static constexpr int kTotal = kUsed > 120 * 1024 ? kUsed : 120 * 1024;      // one CTA per SM: it takes all of the tensor memory
};

template <int DV, bool FULL>
__device__ __forceinline__ void softmax_tile(uint32_t t_s, uint32_t t_o, float scale_log2, int lo, int hi, bool have_o, float& m_used, float& l) {
  uint32_t sa[32];
  float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll 1
  for (int c = 0; c < 4; ++c) {
    tmem_ld_32x32(t_s + 32 * c, sa);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      const float v = __uint_as_float(sa[i]) * scale_log2;
      if (FULL || (32 * c + i >= lo && 32 * c + i < hi)) mx[i & 3] = fmaxf(mx[i & 3], v);
    }
  }
  // a row keeps its old reference unless the new maximum is far above it; the decision is per warp because the tensor
  // memory accesses of the rescale are warp-wide
  const float m4 = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
  const bool warp_grow = __any_sync(0xffffffffu, m4 > m_used + kLazyRescale || (m_used == -INFINITY && m4 > -INFINITY));
  float corr = 1.f;
  if (warp_grow) {
    const float m_new = fmaxf(m_used, m4);
    corr = m_new == -INFINITY ? 1.f : ex2(m_used - m_new);
    m_used = m_new;
    l *= corr;
  }
  const float m_ref = m_used == -INFINITY ? 0.f : m_used;
  float sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 1
  for (int c = 0; c < 4; ++c) {
    tmem_ld_32x32(t_s + 32 * c, sa);
    tmem_ld_wait();
    uint32_t ph[16], pl[16];
#pragma unroll
    for (int i = 0; i < 32; i += 2) {
      float v[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        v[e] = ex2(fmaf(__uint_as_float(sa[i + e]), scale_log2, -m_ref));
        if (!FULL && (32 * c + i + e < lo || 32 * c + i + e >= hi)) v[e] = 0.f;
        sum[(i + e) & 3] += v[e];
      }
      const uint32_t h = pack_bf16x2(v[0], v[1]);
      const float2 back = unpack_bf16x2(h);
      ph[i / 2] = h;
      pl[i / 2] = pack_bf16x2(v[0] - back.x, v[1] - back.y);
    }
    tmem_st_32x16(t_s + 32 * c, ph);
    tmem_st_32x16(t_s + 32 * c + 16, pl);
  }
  l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
  if (warp_grow && have_o) {
#pragma unroll 1
    for (int c = 0; c < DV / 32; ++c) {
      tmem_ld_32x32(t_o + 32 * c, sa);
      tmem_ld_wait();
      uint32_t a[16], b[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        a[i] = __float_as_uint(__uint_as_float(sa[i]) * corr);
        b[i] = __float_as_uint(__uint_as_float(sa[16 + i]) * corr);
      }
      tmem_st_32x16(t_o + 32 * c, a);
      tmem_st_32x16(t_o + 32 * c + 16, b);
    }
  }
  tmem_st_wait();
}

// columns [c0, c0 + 32) of an output row
__device__ __forceinline__ void store_32(const Maps& p, bf16* dst, int c0, const float (&y)[32]) {
  if (p.vec) {
#pragma unroll
    for (int i = 0; i < 32; i += 8) {
      if (c0 + i >= p.v_dim) continue;
      uint4 w;
      w.x = pack_bf16x2(y[i], y[i + 1]), w.y = pack_bf16x2(y[i + 2], y[i + 3]), w.z = pack_bf16x2(y[i + 4], y[i + 5]), w.w = pack_bf16x2(y[i + 6], y[i + 7]);
      *reinterpret_cast<uint4*>(dst + c0 + i) = w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (c0 + i < p.v_dim) dst[c0 + i] = __float2bfloat16(y[i]);
  }
}

__device__ __forceinline__ void softmax_barrier() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

template <int DK, int DV, int M>
__global__ void __launch_bounds__(kThreads, 1) maps_prefill_kernel(const __grid_constant__ CUtensorMap tma_k, const __grid_constant__ CUtensorMap tma_v,
                                                                   const Maps p, int min_rows) {
  using L = PrefillTile<DK, DV, M>;
  constexpr int TBK = tile_bytes<DK>(), TBV = tile_bytes<DV>(), NST = L::kStages, CTA_ROWS = M == 2 ? kRows : 2 * kRows;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sq = smem;                                                // one tile per stream
  uint8_t* sk = smem + L::kQ;                                        // [stage][map]
  uint8_t* sv = sk + NST * L::kK;                                    // [stage]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sv + NST * L::kV);
  uint64_t *k_full = bars, *k_empty = bars + 2, *v_full = bars + 4, *v_empty = bars + 6;      // [stage]
  uint64_t *s_full = bars + 8, *p_ready = bars + 10, *o_done = bars + 12;                     // [stream], [stream], one
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 14);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* swap_l = reinterpret_cast<float*>(bars + 32);               // [stream][row] sums of weights, then of squares
  float* swap_ss = swap_l + 2 * kRows;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row0 = (gridDim.x - 1 - blockIdx.x) * CTA_ROWS;          // the tiles with the longest key range start first
  const int kvh = blockIdx.y, seq = blockIdx.z;
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0;
  const int all_rows = qn * p.group;
  if (all_rows < min_rows || row0 >= all_rows) return;
  const int kv_len = p.positions[q0 + qn - 1] + 1, first_pos = kv_len - qn;
  const int last_row = min(row0 + CTA_ROWS, all_rows) - 1;
  const int begin = first_key(p, first_pos + row0 / p.group + 1) / kPage * kPage;
  const int n_tiles = (first_pos + last_row / p.group + 1 - begin + kTile - 1) / kTile;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1), mbar_init(&k_empty[i], 1), mbar_init(&v_full[i], 1), mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1), mbar_init(&p_ready[i], 4);
    }
    mbar_init(o_done, 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 0 && lane == 0) tma_prefetch_desc(&tma_k), tma_prefetch_desc(&tma_v);
  if (warp == 1) tmem_alloc(tmem_slot, 512), tmem_relinquish();
  // query rows -> shared memory in the layout TMA's 128-byte swizzle would have produced
  for (int i = threadIdx.x; i < 2 * kRows * (DK / 8); i += kThreads) {
    const int s = i / (kRows * (DK / 8)), r = i / (DK / 8) % kRows, c = i % (DK / 8);
    const int row = M == 2 ? row0 + r : row0 + s * kRows + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row < all_rows) {
      const long long head = (long long)(q0 + row / p.group) * p.H + kvh * p.group + row % p.group;
      v = *reinterpret_cast<const uint4*>(p.q + (M == 2 ? head * 2 + s : head) * DK + c * 8);
    }
    *reinterpret_cast<uint4*>(sq + s * TBK + (c >> 3) * kHalf + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v;
  }
  fence_proxy_async_smem();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      const int* table = p.block_tables + (size_t)seq * p.max_blocks;
      const int last = (kv_len - 1) / kPage * kPage;                 // pages past the sequence repeat its last one (finite values)
      for (int it = 0; it < n_tiles; ++it) {
        const int b = it % NST, use = it / NST;
        int tok[kTile / kPage];
#pragma unroll
        for (int pg = 0; pg < kTile / kPage; ++pg) tok[pg] = min(begin + it * kTile + pg * kPage, last);
        if (use > 0 && !mbar_wait(&k_empty[b], (use - 1) & 1, abort_flag)) break;
        mbar_expect_tx(&k_full[b], M * TBK);
#pragma unroll
        for (int a = 0; a < M; ++a)
#pragma unroll
          for (int pg = 0; pg < kTile / kPage; ++pg) {
            const int row = page_row(p, table, tok[pg], p.G * M, kvh * M + a);
#pragma unroll
            for (int h = 0; h < DK / 64; ++h) tma_load_2d(sk + b * L::kK + a * TBK + h * kHalf + pg * (kPage * 128), &tma_k, &k_full[b], 64 * h, row);
          }
        if (use > 0 && !mbar_wait(&v_empty[b], (use - 1) & 1, abort_flag)) break;
        mbar_expect_tx(&v_full[b], TBV);
#pragma unroll
        for (int pg = 0; pg < kTile / kPage; ++pg) {
          const int row = page_row(p, table, tok[pg], p.G, kvh);
#pragma unroll
          for (int h = 0; h < DV / 64; ++h) tma_load_2d(sv + b * L::kV + h * kHalf + pg * (kPage * 128), &tma_v, &v_full[b], 64 * h, row);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(128, 128, 1, 1);
      constexpr uint32_t idesc_pv = make_idesc(128, DV, 1, 1) | (1u << 16);      // B is MN-major
      const uint32_t q_addr = smem_u32(sq), k_addr = smem_u32(sk), v_addr = smem_u32(sv);
      auto scores = [&](int it, int s) {
        const uint32_t qb = q_addr + s * TBK, kb = k_addr + (it % NST) * L::kK + (M == 2 ? s * TBK : 0);
#pragma unroll
        for (int k = 0; k < DK / 16; ++k) {
          const uint32_t off = (k >> 2) * kHalf + (k & 3) * 32;
          tc_mma_bf16(tmem_base + 128 * s, make_smem_desc_sw128(qb + off), make_smem_desc_sw128(kb + off), idesc_s, k > 0);
        }
        tc_commit(&s_full[s]);
        if (s == 1) tc_commit(&k_empty[it % NST]);
      };
      bool ok = mbar_wait(&k_full[0], 0, abort_flag);
      if (ok) {
        tc_fence_after_sync();
        scores(0, 0);
        scores(0, 1);
      }
      for (int it = 0; ok && it < n_tiles; ++it) {
        const int b = it % NST, nb = (it + 1) % NST;
        if (!(ok = mbar_wait(&v_full[b], (it / NST) & 1, abort_flag))) break;
#pragma unroll
        for (int s = 0; s < 2; ++s) {
          if (!(ok = mbar_wait(&p_ready[s], it & 1, abort_flag))) break;
          tc_fence_after_sync();
          const uint32_t t_s = tmem_base + 128 * s, t_o = tmem_base + 256 + 128 * s;
#pragma unroll
          for (int k = 0; k < kTile / 16; ++k) {
            const uint32_t a = t_s + 32 * (k >> 1) + 8 * (k & 1);
            const uint64_t v = desc_mn_major<DV>(v_addr + b * L::kV + k * 2048);
            tc_mma_bf16_ts(t_o, a, v, idesc_pv, it > 0 || k > 0);
            tc_mma_bf16_ts(t_o, a + 16, v, idesc_pv, 1);
          }
          if (s == 1) tc_commit(&v_empty[b]);
          if (it + 1 < n_tiles) {
            if (s == 0) {
              if (!(ok = mbar_wait(&k_full[nb], ((it + 1) / NST) & 1, abort_flag))) break;
              tc_fence_after_sync();
            }
            scores(it + 1, s);
          } else if (s == 1) {
            tc_commit(o_done);
          }
        }
      }
    }
  } else {
    const int s = (warp - 2) >> 2, r = (warp & 3) * 32 + lane;       // stream, and the row in the lane quarter this warp may touch
    const uint32_t lane_off = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t t_s = tmem_base + 128 * s + lane_off, t_o = tmem_base + 256 + 128 * s + lane_off;
    const int srow0 = M == 2 ? row0 : row0 + s * kRows, n_rows = max(0, min(kRows, all_rows - srow0));
    const bool valid = r < n_rows;
    const int lim = valid ? first_pos + (srow0 + r) / p.group + 1 : 0, beg = first_key(p, lim);
    const int lim_first = first_pos + srow0 / p.group + 1, beg_last = first_key(p, first_pos + (srow0 + kRows - 1) / p.group + 1);
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int it = 0; it < n_tiles; ++it) {
      const int tok0 = begin + it * kTile;
      if (!mbar_wait(&s_full[s], it & 1, abort_flag)) { ok = false; break; }
      tc_fence_after_sync();
      if (n_rows == kRows && tok0 + kTile <= lim_first && tok0 >= beg_last)      // every row of the stream sees the whole tile
        softmax_tile<DV, true>(t_s, t_o, p.scale_log2, 0, 0, it > 0, m_used, l);
      else
        softmax_tile<DV, false>(t_s, t_o, p.scale_log2, beg - tok0, lim - tok0, it > 0, m_used, l);
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready[s]);
    }
    ok = ok && mbar_wait(o_done, 0, abort_flag);
    tc_fence_after_sync();
    const int row = srow0 + r;
    bf16* dst = p.out + (long long)(q0 + row / p.group) * p.ldo + (long long)(kvh * p.group + row % p.group) * p.v_dim;
    if (M == 2) {
      // both groups of warps take half of the columns of the combined row
      constexpr int N = DV / 64;                                     // 32-column pieces per group
      swap_l[s * kRows + r] = l;
      softmax_barrier();
      const float l0 = swap_l[r], l1 = swap_l[kRows + r];
      const float i0 = l0 > 0.f ? 1.f / l0 : 0.f, i1 = l1 > 0.f ? p.lam / l1 : 0.f;
      float y[N][32], ss = 0.f;
#pragma unroll
      for (int n = 0; n < N; ++n) {
        const uint32_t col = tmem_base + 256 + lane_off + (s * N + n) * 32;
        uint32_t a[32], b[32];
        tmem_ld_32x32(col, a);
        tmem_ld_32x32(col + 128, b);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          y[n][i] = __uint_as_float(a[i]) * i0 - __uint_as_float(b[i]) * i1;
          ss = fmaf(y[n][i], y[n][i], ss);
        }
      }
      swap_ss[s * kRows + r] = ss;
      softmax_barrier();
      const float f = p.out_scale / sqrtf((swap_ss[r] + swap_ss[kRows + r]) / (float)p.v_dim + p.eps);
      if (ok && valid) {
#pragma unroll
        for (int n = 0; n < N; ++n) {
#pragma unroll
          for (int i = 0; i < 32; ++i) y[n][i] *= f;
          store_32(p, dst, (s * N + n) * 32, y[n]);
        }
      }
    } else if (ok) {
      if (valid) l += sink_weight(p, kvh * p.group + row % p.group, m_used);
      const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll 1
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t a[32];
        tmem_ld_32x32(t_o + 32 * c, a);
        tmem_ld_wait();
        if (!valid) continue;
        float y[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) y[i] = __uint_as_float(a[i]) * inv;
        store_32(p, dst, 32 * c, y);
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) { tc_fence_after_sync(); tmem_dealloc(tmem_base, 512); }
  if (threadIdx.x == 0 && *abort_flag && p.status) atomicCAS(p.status, FLLM_OK, FLLM_ERR_MBAR_TIMEOUT);
}

// ------------------------------------------------------------------------------------------ host
template <int DK, int DV, int M>
int launch_tc(Maps a, const MapsAttnParams& p, int splits, cudaStream_t s) {
  using D = DecodeTile<DK, DV, M>;
  using P = PrefillTile<DK, DV, M>;
  static bool configured[kMaxDevices] = {};
  if (first_call_on_device(configured)) {
    cuda_check(cudaFuncSetAttribute(maps_decode_kernel<DK, DV, M>, cudaFuncAttributeMaxDynamicSharedMemorySize, D::kTotal), "maps_decode smem");
    cuda_check(cudaFuncSetAttribute(maps_prefill_kernel<DK, DV, M>, cudaFuncAttributeMaxDynamicSharedMemorySize, P::kTotal), "maps_prefill smem");
  }
  int launches = 0;
  const int max_rows = p.max_q_len * a.group;
  if (p.min_q_len * a.group <= kDecodeRows) {
    a.splits = max_rows <= kDecodeRows ? splits : 1;      // partial results of longer sequences do not exist
    const int row_tiles = (std::min(max_rows, kDecodeRows) + D::kRowsOf - 1) / D::kRowsOf;
    launch_pdl(maps_decode_kernel<DK, DV, M>, dim3(a.G * row_tiles, p.num_seqs, a.splits), dim3(128), D::kTotal, s, a, row_tiles, (int)kDecodeRows);
    ++launches;
    if (a.splits > 1) {
      launch_pdl(maps_merge_kernel<DV, M>, dim3((p.tokens * a.H + 3) / 4), dim3(128), 0, s, a, p.tokens);
      ++launches;
    }
  }
  if (max_rows > kDecodeRows) {
    constexpr int rows = M == 2 ? kRows : 2 * kRows;
    const uint64_t n = (uint64_t)p.num_blocks * a.G * a.block_size;
    // (copies: a second lookup may move the first entry)
    const CUtensorMap km = pool_map(p.k_cache, n * M, DK), vm = pool_map(p.v_cache, n, DV);
    maps_prefill_kernel<DK, DV, M><<<dim3((max_rows + rows - 1) / rows, a.G, p.num_seqs), kThreads, P::kTotal, s>>>(km, vm, a, kDecodeRows + 1);
    ++launches;
  }
  cuda_check(cudaGetLastError(), "attention_maps launch");
  return launches;
}

template <typename T, int M>
void launch_simple(const MapsAttnParams& p, cudaStream_t s) {
  constexpr int NW = 4;
  const int piece = std::min(p.v_dim, 512), widest = p.spread ? piece : std::max(p.dim, p.v_dim);
  const size_t smem = (size_t)(M * p.dim + M * NW * piece + M * 2 * NW) * sizeof(float);
  const dim3 grid(p.H, p.tokens, p.spread ? (p.v_dim + 511) / 512 : 1);
  if (widest <= 64) maps_simple_kernel<T, 2, M, NW><<<grid, NW * 32, smem, s>>>(p);
  else if (widest <= 128) maps_simple_kernel<T, 4, M, NW><<<grid, NW * 32, smem, s>>>(p);
  else if (widest <= 256) maps_simple_kernel<T, 8, M, NW><<<grid, NW * 32, smem, s>>>(p);
  else if (widest <= 512) maps_simple_kernel<T, 16, M, NW><<<grid, NW * 32, smem, s>>>(p);
  else throw std::runtime_error("attention_maps: heads of at most 512 values");
  cuda_check(cudaGetLastError(), "maps_simple_kernel");
}

}  // namespace

bool attention_maps_tc_supported(int wk, int wv, int block_size, int f32) {
  return !f32 && (wk == 64 || wk == 128) && (wv == 64 || wv == 128) && block_size % kPage == 0;
}
// key slices the tensor-core path uses for a step (1: no workspace needed)
int attention_maps_splits(int num_seqs, int max_q_len, int H, int G, int maps, int max_kv_len, int window) {
  const int rows = max_q_len * (H / G), per_tile = 16 / maps;
  if (rows > kDecodeRows) return 1;
  const long long ctas = (long long)num_seqs * G * ((rows + per_tile - 1) / per_tile);
  const int keys = window > 0 ? std::min(max_kv_len, window + max_q_len) : max_kv_len, pages = (keys + kPage - 1) / kPage;
  if (ctas >= sm_count()) return 1;
  return std::max(1, (int)std::min<long long>({(2 * sm_count() + ctas - 1) / ctas, (pages + 7) / 8, 32}));
}
size_t attention_maps_workspace_bytes(int tokens, int q_heads, int wv, int splits) {
  return splits > 1 ? (size_t)tokens * q_heads * splits * (wv + 2) * sizeof(float) : 0;
}

int attention_maps(const MapsAttnParams& p, int splits, void* workspace, size_t workspace_bytes, bool tensor_cores, int* status, cudaStream_t s) {
  if (p.tokens <= 0) return 0;
  if (p.tokens > 65535 || p.num_seqs > 65535) throw std::runtime_error("attention_maps: at most 65535 rows and sequences in a step");
  if (p.maps != 1 && p.maps != 2) throw std::runtime_error("attention_maps: one or two maps");
  if (p.maps == 2 && (p.sink || p.r1 || p.spread)) throw std::runtime_error("attention_maps: sinks, distance biases and spread values go with one map");
  if (p.spread && (!p.part_o || !p.part_ml)) throw std::runtime_error("attention_maps: spread values need room for partial sums");
  const bool fast = p.spread ? attention_spread_tc_supported(p.H / p.G, p.wk, p.wv, p.block_size, p.f32) && p.scale > 0.f && p.bias_range <= kTalkBiasRange
                             : !p.r1 && attention_maps_tc_supported(p.wk, p.wv, p.block_size, p.f32);
  if (!tensor_cores || !fast) {
    if (p.spread && splits > 1) throw std::runtime_error("attention_maps: key slices are the tensor-core path's");
    if (p.f32) p.maps == 2 ? launch_simple<float, 2>(p, s) : launch_simple<float, 1>(p, s);
    else p.maps == 2 ? launch_simple<bf16, 2>(p, s) : launch_simple<bf16, 1>(p, s);
    return 1;
  }
  if (p.spread) return attention_spread_tc(p, splits, status, s);
  splits = std::max(splits, 1);
  if (workspace_bytes < attention_maps_workspace_bytes(p.tokens, p.H * p.maps, p.wv, splits))
    throw std::runtime_error("attention_maps: workspace too small for the requested key slices");
  Maps a{};
  a.q = static_cast<const bf16*>(p.q), a.kc = static_cast<const bf16*>(p.k_cache), a.vc = static_cast<const bf16*>(p.v_cache);
  a.block_tables = p.block_tables, a.max_blocks = p.max_blocks, a.q_starts = p.q_starts, a.positions = p.positions;
  a.out = static_cast<bf16*>(p.out), a.ldo = p.ldo;
  a.H = p.H, a.G = p.G, a.group = p.H / p.G, a.v_dim = p.v_dim, a.block_size = p.block_size;
  a.vec = p.v_dim % 8 == 0 && p.ldo % 8 == 0 && (reinterpret_cast<uintptr_t>(p.out) & 15) == 0;
  a.window = p.window, a.scale_log2 = p.scale * kLog2e, a.lam = p.lam, a.out_scale = p.out_scale, a.eps = p.eps;
  a.ws_o = static_cast<float*>(workspace);
  a.ws_ml = a.ws_o != nullptr ? a.ws_o + (size_t)p.tokens * p.H * p.maps * splits * p.wv : nullptr;
  a.status = status;
  a.sink = p.sink;
#define FLLM_MAPS(K_, V_) return p.maps == 2 ? launch_tc<K_, V_, 2>(a, p, splits, s) : launch_tc<K_, V_, 1>(a, p, splits, s);
  if (p.wk == 64 && p.wv == 64) { FLLM_MAPS(64, 64) }
  if (p.wk == 64) { FLLM_MAPS(64, 128) }
  if (p.wv == 64) { FLLM_MAPS(128, 64) }
  FLLM_MAPS(128, 128)
#undef FLLM_MAPS
}

void maps_prepare(const MapsPrepareParams& params, cudaStream_t s) {
  if (params.tokens <= 0) return;
  MapsPrepareParams p = params;
  if (p.taps > kMaxTaps || (p.taps > 0 && (p.conv_width % 4 || reinterpret_cast<uintptr_t>(p.conv_w) % 16 || reinterpret_cast<uintptr_t>(p.conv_state) % 16)))
    throw std::runtime_error("maps_prepare: a convolution of at most 8 taps, columns in multiples of 4");
  if (p.taps > 0 && p.full) throw std::runtime_error("maps_prepare: a norm over all maps does not go with a convolution");
  const uintptr_t any = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.bias) | reinterpret_cast<uintptr_t>(p.partials);
  p.vec = p.dim % 4 == 0 && p.v_dim % 4 == 0 && p.q_offset % 4 == 0 && p.k_offset % 4 == 0 && p.v_offset % 4 == 0 && any % 16 == 0 &&
          (p.partials ? p.width % 4 == 0 && p.plane % 4 == 0 : p.ldx % 4 == 0);
  const uintptr_t norms = reinterpret_cast<uintptr_t>(p.q_norm) | reinterpret_cast<uintptr_t>(p.k_norm);
  p.lanes = p.vec && (p.wk == 64 || p.wk == 128) && (p.pairs ? p.rot % 4 == 0 : p.rot % 8 == 0) && norms % 16 == 0 ? p.wk / 4 : 0;
  const int heads = p.q_heads + p.k_heads + p.v_heads;
  const int shares = std::max(1, std::min((heads + 3) / 4, 4 * sm_count() / std::max(p.tokens, 1)));
  const size_t smem = (size_t)(p.rot + 4 * p.dim) * sizeof(float);
  if (smem > 48 * 1024) throw std::runtime_error("maps_prepare: heads too wide");
  const dim3 grid(p.tokens, shares);
  if (p.taps > 0) {
    if (p.f32) launch_pdl(maps_prepare_kernel<float, true>, grid, dim3(128), smem, s, p);
    else launch_pdl(maps_prepare_kernel<bf16, true>, grid, dim3(128), smem, s, p);
  } else {
    if (p.f32) launch_pdl(maps_prepare_kernel<float, false>, grid, dim3(128), smem, s, p);
    else launch_pdl(maps_prepare_kernel<bf16, false>, grid, dim3(128), smem, s, p);
  }
  cuda_check(cudaGetLastError(), "maps_prepare_kernel");
}

}  // namespace fllm
