// Attention whose values are the keys themselves ("tied"): a token caches one row per key/value head, the projected key, and
// one fp32 factor. The factor (for instance the reciprocal root mean square of the key) multiplies the key where it meets a
// query and not where it serves as value, and every query head has an fp32 factor of its own (norm, temperature, softmax
// scale), so normalised keys and queries are never rounded and the cache is half the size of separate keys and values:
//   s = (q . k_j) qf f_j;  with a cap c > 0: s <- c tanh(s / c);  out = softmax(s) k
// Row length W is the head width padded with zeros (64, 128, or a multiple of 16 above); pool [block][kv head][token][W],
// factors [block][kv head][token]. Query rows of a sequence are numbered token * group + head within one kv head.
//
//   tied_prefill_kernel  tcgen05 with accumulators in tensor memory, 128 query rows per CTA, W = 64 or 128: one K tile in shared
//                        memory is the K-major operand of S = Q K^T and the MN-major operand of O += P K.
//   tied_decode_kernel   mma.sync, 16 query rows per CTA (sequences with few query rows are bound by the cache reads), each warp
//                        streaming its own 16-token pages through a private cp.async ring; split over key slices.
//   tied_simple_kernel   CUDA cores, any width, bf16 and fp32.
//
// Weights are fp32; for the tensor-core product with the values a weight travels as the sum of two bf16 values (16 significant
// bits). A cap of at most kFixedCap bounds every score, so the softmax needs no running maximum and no rescaling: its
// reference is zero, exp(+-64) and sums over any context stay far inside the fp32 range.
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
constexpr float kFixedCap = 64.f;
constexpr int kDecodeRows = 64;           // sequences with at most this many query rows per kv head run in the decode kernel

__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ------------------------------------------------------------------------------------------ factors and cache rows
// One warp per (token, head), query heads first. Query head: q_factor[t][h] = scale * temperature(position) / rms(q). Key head:
// the row goes to the cache with f = 1 / rms(k). rms(x) = sqrt(mean x^2 + eps); eps < 0: no norm (factor 1). temperature =
// 1 + coef ln(floor((position + 1) / every) + 1). With split-K partial sums as the source, queries are also written to q_out.
template <typename T>
__global__ void __launch_bounds__(128) tied_prepare_kernel(const TiedPrepareParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int item = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int heads = p.H + p.G;
  if (item >= p.tokens * heads) return;
  const int t = item / heads, h = item - t * heads;
  const bool is_q = h < p.H;
  const int col = is_q ? h * p.dim : p.k_offset + (h - p.H) * p.dim;
  const T* src = static_cast<const T*>(p.x) + (long long)t * p.ldx + col;
  const float* part = p.partials ? p.partials + (size_t)t * p.width + col : nullptr;
  const int slot = is_q ? 0 : p.slots[t];
  if (slot < 0) return;
  T* dst = nullptr;                                        // where the (rounded) values go
  if (!is_q) dst = static_cast<T*>(p.cache) + (((long long)(slot / p.block_size) * p.G + (h - p.H)) * p.block_size + slot % p.block_size) * p.W;
  else if (part) dst = static_cast<T*>(p.q_out) + (long long)t * p.ld_qout + h * p.dim;
  float ss = 0.f;
  if (p.vec) {                                             // four values per lane
    using V4 = typename Four<T>::type;
    for (int c = 4 * lane; c < p.dim; c += 128) {
      V4 raw;
      T* v = reinterpret_cast<T*>(&raw);
      if (part) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s = 0; s < p.splits; ++s) {
          const float4 q = __ldcg(reinterpret_cast<const float4*>(part + s * p.plane + c));
          acc.x += q.x, acc.y += q.y, acc.z += q.z, acc.w += q.w;
        }
        v[0] = from_f32<T>(acc.x), v[1] = from_f32<T>(acc.y), v[2] = from_f32<T>(acc.z), v[3] = from_f32<T>(acc.w);
      } else {
        raw = *reinterpret_cast<const V4*>(src + c);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) ss = fmaf(to_f32(v[e]), to_f32(v[e]), ss);
      if (dst) *reinterpret_cast<V4*>(dst + c) = raw;
    }
  } else {
    for (int c = lane; c < p.dim; c += 32) {
      T v;
      if (part) {
        float acc = 0.f;
        for (int s = 0; s < p.splits; ++s) acc += __ldcg(part + s * p.plane + c);
        v = from_f32<T>(acc);
      } else {
        v = src[c];
      }
      ss = fmaf(to_f32(v), to_f32(v), ss);
      if (dst) dst[c] = v;
    }
  }
  if (!is_q)
    for (int c = p.dim + lane; c < p.W; c += 32) dst[c] = from_f32<T>(0.f);
  ss = warp_sum(ss);
  if (lane != 0) return;
  const float inv = p.eps >= 0.f ? 1.f / sqrtf(ss / (float)p.dim + p.eps) : 1.f;
  if (is_q) {
    float f = p.scale * inv;
    if (p.temp_coef != 0.f) f *= 1.f + p.temp_coef * logf(floorf((float)(p.positions[t] + 1) / p.temp_every) + 1.f);
    p.q_factor[(long long)t * p.H + h] = f;
  } else {
    p.key_factor[((long long)(slot / p.block_size) * p.G + (h - p.H)) * p.block_size + slot % p.block_size] = inv;
  }
}

// ------------------------------------------------------------------------------------------ CUDA-core attention
// One CTA per (head, token); its warps take every NW-th key with an online softmax each and are merged through shared memory.
template <typename T, int EV, int NW>
__global__ void __launch_bounds__(NW * 32) tied_simple_kernel(const TiedAttnParams p) {
  extern __shared__ float sm[];
  float* sq = sm;                              // [dim] query row * factor
  float* sacc = sq + p.dim;                    // [NW][dim]
  float* sml = sacc + NW * p.dim;              // [NW][2] maximum and sum
  const int h = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (p.H / p.G);
  const T* q = static_cast<const T*>(p.q) + (long long)t * p.ldq + h * p.dim;
  const T* cache = static_cast<const T*>(p.cache);
  const float qf = p.q_factor[(long long)t * p.H + h];
  for (int i = threadIdx.x; i < p.dim; i += NW * 32) sq[i] = to_f32(q[i]);
  __syncthreads();
  const int kv_len = p.positions[t] + 1;
  const int* table = p.block_tables + (size_t)p.row_seq[t] * p.max_blocks;
  float m = -INFINITY, l = 0.f, acc[EV];
#pragma unroll
  for (int e = 0; e < EV; ++e) acc[e] = 0.f;
  for (int j = warp; j < kv_len; j += NW) {
    const size_t at = ((size_t)table[j / p.block_size] * p.G + g) * p.block_size + j % p.block_size;
    const T* row = cache + at * p.W;
    float s = 0.f, v[EV];
#pragma unroll
    for (int e = 0; e < EV; ++e) {
      const int c = lane + 32 * e;
      v[e] = c < p.dim ? to_f32(row[c]) : 0.f;
      if (c < p.dim) s = fmaf(v[e], sq[c], s);
    }
    s = warp_sum(s) * (qf * p.key_factor[at]);
    if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    const float mn = fmaxf(m, s), corr = expf(m - mn), pr = expf(s - mn);
    l = l * corr + pr;
#pragma unroll
    for (int e = 0; e < EV; ++e) acc[e] = fmaf(acc[e], corr, pr * v[e]);
    m = mn;
  }
#pragma unroll
  for (int e = 0; e < EV; ++e)
    if (lane + 32 * e < p.dim) sacc[warp * p.dim + lane + 32 * e] = acc[e];
  if (lane == 0) sml[2 * warp] = m, sml[2 * warp + 1] = l;
  __syncthreads();
  float mm = -INFINITY;
#pragma unroll
  for (int w = 0; w < NW; ++w) mm = fmaxf(mm, sml[2 * w]);
  float c[NW], tot = 0.f;
#pragma unroll
  for (int w = 0; w < NW; ++w) {
    c[w] = sml[2 * w] == -INFINITY ? 0.f : expf(sml[2 * w] - mm);
    tot = fmaf(sml[2 * w + 1], c[w], tot);
  }
  T* out = static_cast<T*>(p.out) + (long long)t * p.ldo + h * p.dim;
  for (int i = threadIdx.x; i < p.dim; i += NW * 32) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) v = fmaf(sacc[w * p.dim + i], c[w], v);
    out[i] = from_f32<T>(v / tot);
  }
}

// ------------------------------------------------------------------------------------------ shared by the tensor-core kernels
struct Tied {
  const bf16* q;
  long long ldq;
  const float* q_factor;
  const bf16* cache;
  const float* key_factor;
  const int* block_tables;
  int max_blocks;
  const int *q_starts, *positions;
  bf16* out;
  long long ldo;
  int H, G, group, dim, block_size, vec;     // vec: rows of q and out can be moved in 16-byte pieces
  float softcap;
  float *ws_o, *ws_ml;                       // partial results of key slices: [T][H][splits][D], [T][H][splits][2]
  int splits;
  int* status;
};

// Score in the exp2 domain. `f` = product of the factors, times 2 log2(e) / cap under a cap and log2(e) without.
template <bool CAP>
__device__ __forceinline__ float log2_score(float acc, float f, float cap2) {
  if (!CAP) return acc * f;
  return fmaf(-2.f * cap2, rcp(1.f + ex2(acc * f)), cap2);        // cap2 tanh(x) = cap2 - 2 cap2 / (1 + e^(2x))
}
template <bool CAP>
__device__ __forceinline__ float row_factor(const Tied& p, int t, int h) {
  return p.q_factor[(long long)t * p.H + h] * (CAP ? 2.f * kLog2e / p.softcap : kLog2e);
}

// 16-byte piece c (columns 8c .. 8c + 7) of a query row, zeros beyond the head's width
__device__ __forceinline__ uint4 query_piece(const Tied& p, int t, int h, int c) {
  const bf16* src = p.q + (long long)t * p.ldq + (long long)h * p.dim + c * 8;
  if (p.vec) return c * 8 < p.dim ? *reinterpret_cast<const uint4*>(src) : make_uint4(0, 0, 0, 0);
  __align__(16) bf16 v[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) v[i] = c * 8 + i < p.dim ? src[i] : __float2bfloat16(0.f);
  return *reinterpret_cast<const uint4*>(v);
}

// first pool row of the kPage tokens from `token` on
__device__ __forceinline__ int page_row(const Tied& p, const int* table, int token, int kvh) {
  return (table[token / p.block_size] * p.G + kvh) * p.block_size + token % p.block_size;
}

// ------------------------------------------------------------------------------------------ decode
template <int D>
struct DecodeTile {
  static constexpr int kStages = 4;
  static constexpr int kRowBytes = kPage * D * 2, kStage = kRowBytes + kPage * 4;      // key rows, then their factors
  static constexpr int kQ = 16 * D * 2, kRing = 4 * kStages * kStage;
  static constexpr int kMerge = 4 * 16 * D * 4 + 4 * 16 * 2 * 4;
  static constexpr int kTotal = kQ + (kRing > kMerge ? kRing : kMerge) + 128;
};

// FIXED: the cap bounds the scores, reference 0; otherwise a running maximum
template <int D, bool CAP, bool FIXED>
__global__ void __launch_bounds__(128, 3) tied_decode_kernel(const Tied p, int row_tiles, int max_rows) {
  using L = DecodeTile<D>;
  extern __shared__ __align__(128) uint8_t smem[];
  bf16* qtile = reinterpret_cast<bf16*>(smem);
  uint8_t* ring = smem + L::kQ;
  const int kvh = blockIdx.x / row_tiles, row0 = (blockIdx.x % row_tiles) * 16, seq = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0;
  const int all_rows = qn * p.group;
  if (qn <= 0 || all_rows > max_rows || row0 >= all_rows) return;
  const int n_rows = min(16, all_rows - row0);
  const int kv_len = p.positions[q0 + qn - 1] + 1, first_pos = kv_len - qn;
  const int hi_tok = first_pos + (row0 + n_rows - 1) / p.group + 1;
  const int pages = (hi_tok + kPage - 1) / kPage;
  const int per = (pages + p.splits - 1) / p.splits;
  const int pg0 = split * per, pg1 = min(pg0 + per, pages);

  for (int i = threadIdx.x; i < 16 * (D / 8); i += 128) {
    const int r = i / (D / 8), c = i - r * (D / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < n_rows) v = query_piece(p, q0 + (row0 + r) / p.group, kvh * p.group + (row0 + r) % p.group, c);
    *reinterpret_cast<uint4*>(tile_ptr<D>(qtile, r, c)) = v;
  }
  __syncthreads();
  uint32_t qf[D / 16][4];
#pragma unroll
  for (int kk = 0; kk < D / 16; ++kk) ldsm_x4(qf[kk], tile_ptr<D>(qtile, lane & 15, 2 * kk + (lane >> 4)));

  const int g = lane >> 2, t4 = lane & 3;
  int lim[2];
  float rf[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = g + 8 * i;
    lim[i] = 0, rf[i] = 0.f;
    if (r < n_rows) {
      lim[i] = first_pos + (row0 + r) / p.group + 1;
      rf[i] = row_factor<CAP>(p, q0 + (row0 + r) / p.group, kvh * p.group + (row0 + r) % p.group);
    }
  }
  const float cap2 = p.softcap * kLog2e;
  float o[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {FIXED ? 0.f : -INFINITY, FIXED ? 0.f : -INFINITY}, l[2] = {0.f, 0.f};

  uint8_t* mine = ring + (size_t)warp * L::kStages * L::kStage;
  const int* table = p.block_tables + (size_t)seq * p.max_blocks;
  auto issue = [&](int it) {
    const int pg = pg0 + warp + 4 * it;
    if (pg < pg1) {
      const long long row = page_row(p, table, pg * kPage, kvh);
      uint8_t* st = mine + (size_t)(it % L::kStages) * L::kStage;
      const bf16* src = p.cache + row * D;
#pragma unroll
      for (int i = lane; i < kPage * (D / 8); i += 32) {
        const int r = i / (D / 8), c = i - r * (D / 8);
        cp_async16(tile_ptr<D>(reinterpret_cast<bf16*>(st), r, c), src + (size_t)r * D + c * 8);
      }
      if (lane < kPage / 4) cp_async16(st + L::kRowBytes + lane * 16, p.key_factor + row + lane * 4);
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
    bf16* ks = reinterpret_cast<bf16*>(st);
    const float* kf = reinterpret_cast<const float*>(st + L::kRowBytes);
    const int tok_base = (pg0 + warp + 4 * it) * kPage, j4 = lane >> 3;
    float s[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t b[4];
      ldsm_x4(b, tile_ptr<D>(ks, (j4 >> 1) * 8 + (lane & 7), 2 * kk + (j4 & 1)));
      mma_bf16(s[0], qf[kk], b[0], b[1]);
      mma_bf16(s[1], qf[kk], b[2], b[3]);
    }
    // ---- weights of two rows x four tokens
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      const float2 f = *reinterpret_cast<const float2*>(kf + nb * 8 + 2 * t4);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float v = log2_score<CAP>(s[nb][e], (e & 1 ? f.y : f.x) * rf[e >> 1], cap2);
        s[nb][e] = tok_base + nb * 8 + 2 * t4 + (e & 1) < lim[e >> 1] ? v : -INFINITY;
        if (!FIXED) mx[e >> 1] = fmaxf(mx[e >> 1], s[nb][e]);
      }
    }
    float ref[2] = {0.f, 0.f};
    if (!FIXED) {
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
        for (int db = 0; db < D / 8; ++db) o[db][2 * i] *= c, o[db][2 * i + 1] *= c;
      }
    }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float p0 = ex2(s[nb][2 * i] - ref[i]), p1 = ex2(s[nb][2 * i + 1] - ref[i]);
        l[i] += p0 + p1;
        const uint32_t hi = pack_bf16x2(p0, p1);
        const float2 back = unpack_bf16x2(hi);
        ph[nb * 2 + i] = hi;
        pl[nb * 2 + i] = pack_bf16x2(p0 - back.x, p1 - back.y);
      }
#pragma unroll
    for (int db = 0; db < D / 8; db += 2) {
      uint32_t b[4];
      ldsm_x4_t(b, tile_ptr<D>(ks, (j4 & 1) * 8 + (lane & 7), db + (j4 >> 1)));
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
  float* mo = reinterpret_cast<float*>(smem + L::kQ);    // [4][16][D]
  float* mml = mo + 4 * 16 * D;                          // [4][16][2]
#pragma unroll
  for (int db = 0; db < D / 8; ++db) {
    *reinterpret_cast<float2*>(mo + ((size_t)warp * 16 + g) * D + db * 8 + 2 * t4) = make_float2(o[db][0], o[db][1]);
    *reinterpret_cast<float2*>(mo + ((size_t)warp * 16 + g + 8) * D + db * 8 + 2 * t4) = make_float2(o[db][2], o[db][3]);
  }
  if (t4 == 0) {
#pragma unroll
    for (int i = 0; i < 2; ++i) mml[(warp * 16 + g + 8 * i) * 2] = m[i], mml[(warp * 16 + g + 8 * i) * 2 + 1] = l[i];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n_rows * D; i += 128) {
    const int r = i / D, d = i - r * D;
    float mm = -INFINITY, ll = 0.f, a = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, mml[(w * 16 + r) * 2]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = mml[(w * 16 + r) * 2];
      const float c = mw == -INFINITY ? 0.f : ex2(mw - mm);
      ll += mml[(w * 16 + r) * 2 + 1] * c;
      a += mo[((size_t)w * 16 + r) * D + d] * c;
    }
    const int head = kvh * p.group + (row0 + r) % p.group;
    const long long tok = q0 + (row0 + r) / p.group;
    if (p.splits == 1) {
      if (d < p.dim) p.out[tok * p.ldo + (long long)head * p.dim + d] = __float2bfloat16(ll > 0.f ? a / ll : 0.f);
    } else {
      const size_t base = ((size_t)tok * p.H + head) * p.splits + split;
      p.ws_o[base * D + d] = a;
      if (d == 0) p.ws_ml[base * 2] = mm, p.ws_ml[base * 2 + 1] = ll;
    }
  }
}

// one warp per (token, head)
template <int D>
__global__ void __launch_bounds__(128) tied_merge_kernel(const Tied p, int T) {
  pdl_launch_dependents();
  pdl_wait();
  const int item = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= T * p.H) return;
  const int tok = item / p.H, head = item - tok * p.H;
  const size_t base = (size_t)item * p.splits;
  float mm = -INFINITY, ll = 0.f, a[D / 32];
  for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, p.ws_ml[(base + s) * 2]);
#pragma unroll
  for (int e = 0; e < D / 32; ++e) a[e] = 0.f;
  for (int s = 0; s < p.splits; ++s) {
    const float ms = p.ws_ml[(base + s) * 2];
    if (ms == -INFINITY) continue;
    const float w = ex2(ms - mm);
    ll = fmaf(p.ws_ml[(base + s) * 2 + 1], w, ll);
#pragma unroll
    for (int e = 0; e < D / 32; ++e) a[e] = fmaf(p.ws_o[(base + s) * D + lane + 32 * e], w, a[e]);
  }
  bf16* dst = p.out + (long long)tok * p.ldo + (long long)head * p.dim;
#pragma unroll
  for (int e = 0; e < D / 32; ++e)
    if (lane + 32 * e < p.dim) dst[lane + 32 * e] = __float2bfloat16(ll > 0.f ? a[e] / ll : 0.f);
}

// ------------------------------------------------------------------------------------------ prefill
// Warp 0 brings K tiles (eight pages of 16 rows by TMA, 128-byte swizzle, plus the tokens' factors) into two stages, warp 1
// issues the MMAs, warps 2 - 5 are the softmax, one thread per query row. The weights of 32 tokens overwrite the 32 columns
// their scores came from: 16 columns of leading bf16 terms, 16 of remainders. Tensor memory: S / P 128 columns, O 128; two
// CTAs share an SM, so one's softmax runs under the other's MMAs. Every wait is bounded.
constexpr int kThreads = 192;
template <int D>
constexpr int prefill_smem() { return 3 * tile_bytes<D>() + 2 * kTile * 4 + 256 + 1024; }

// untiled copy of `bytes` (a multiple of 16, both sides 16-byte aligned) that arrives on a barrier
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes),
               "r"(smem_u32(bar))
               : "memory");
}

template <int D, bool FULL, bool CAP, bool FIXED>
__device__ __forceinline__ void softmax_tile(uint32_t t_s, uint32_t t_o, const float* kf, float rf, float cap2, int hi, bool have_o, float& m_used,
                                             float& l) {
  uint32_t sa[32];
  float m_ref = 0.f, corr = 1.f;
  bool warp_grow = false;
  if (!FIXED) {
    float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll 1
    for (int c = 0; c < 4; ++c) {
      tmem_ld_32x32(t_s + 32 * c, sa);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; i += 4) {
        const float4 f = *reinterpret_cast<const float4*>(kf + 32 * c + i);
        const float fs[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float v = log2_score<CAP>(__uint_as_float(sa[i + e]), fs[e] * rf, cap2);
          if (FULL || 32 * c + i + e < hi) mx[e] = fmaxf(mx[e], v);
        }
      }
    }
    // a row keeps its old reference unless the new maximum is far above it; the decision is per warp because the tensor
    // memory accesses of the rescale are warp-wide
    const float m4 = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
    warp_grow = __any_sync(0xffffffffu, m4 > m_used + kLazyRescale || (m_used == -INFINITY && m4 > -INFINITY));
    if (warp_grow) {
      const float m_new = fmaxf(m_used, m4);
      corr = m_new == -INFINITY ? 1.f : ex2(m_used - m_new);
      m_used = m_new;
      l *= corr;
    }
    m_ref = m_used == -INFINITY ? 0.f : m_used;
  }
  float sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 1
  for (int c = 0; c < 4; ++c) {
    tmem_ld_32x32(t_s + 32 * c, sa);
    tmem_ld_wait();
    uint32_t ph[16], pl[16];
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const float4 f = *reinterpret_cast<const float4*>(kf + 32 * c + i);
      const float fs[4] = {f.x, f.y, f.z, f.w};
      float v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[e] = log2_score<CAP>(__uint_as_float(sa[i + e]), fs[e] * rf, cap2);
        v[e] = ex2(FIXED ? v[e] : v[e] - m_ref);
        if (!FULL && 32 * c + i + e >= hi) v[e] = 0.f;
        sum[e] += v[e];
      }
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const uint32_t h = pack_bf16x2(v[e], v[e + 1]);
        const float2 back = unpack_bf16x2(h);
        ph[(i + e) / 2] = h;
        pl[(i + e) / 2] = pack_bf16x2(v[e] - back.x, v[e + 1] - back.y);
      }
    }
    tmem_st_32x16(t_s + 32 * c, ph);
    tmem_st_32x16(t_s + 32 * c + 16, pl);
  }
  l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
  if (!FIXED && warp_grow && have_o) {
#pragma unroll 1
    for (int c = 0; c < D / 32; ++c) {
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

template <int D, bool CAP, bool FIXED>
__global__ void __launch_bounds__(kThreads, 2) tied_prefill_kernel(const __grid_constant__ CUtensorMap tma_k, const Tied p, int min_rows) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int TB = tile_bytes<D>();
  uint8_t* sq = smem;
  uint8_t* sk = smem + TB;                                           // two stages
  float* skf = reinterpret_cast<float*>(smem + 3 * TB);              // two stages of kTile factors
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + 3 * TB + 2 * kTile * 4);
  uint64_t* k_full = bars;                                           // [2]
  uint64_t* k_empty = bars + 2;                                      // [2]
  uint64_t* s_full = bars + 4;
  uint64_t* p_ready = bars + 5;
  uint64_t* o_done = bars + 6;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row0 = (gridDim.x - 1 - blockIdx.x) * kRows;             // the tiles with the longest key range start first
  const int kvh = blockIdx.y, seq = blockIdx.z;
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0;
  const int all_rows = qn * p.group;
  if (all_rows < min_rows || row0 >= all_rows) return;
  const int n_rows = min(kRows, all_rows - row0);
  const int kv_len = p.positions[q0 + qn - 1] + 1, first_pos = kv_len - qn;
  const int lim_first = first_pos + row0 / p.group + 1, lim_last = first_pos + (row0 + n_rows - 1) / p.group + 1;
  const int n_tiles = (lim_last + kTile - 1) / kTile;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) mbar_init(&k_full[i], 1), mbar_init(&k_empty[i], 1);
    mbar_init(s_full, 1), mbar_init(p_ready, 4), mbar_init(o_done, 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 0 && lane == 0) tma_prefetch_desc(&tma_k);
  if (warp == 1) tmem_alloc(tmem_slot, 256), tmem_relinquish();
  // query rows -> shared memory in the layout TMA's 128-byte swizzle would have produced
  for (int i = threadIdx.x; i < kRows * (D / 8); i += kThreads) {
    const int r = i / (D / 8), c = i % (D / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < n_rows) v = query_piece(p, q0 + (row0 + r) / p.group, kvh * p.group + (row0 + r) % p.group, c);
    *reinterpret_cast<uint4*>(sq + (c >> 3) * kHalf + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v;
  }
  fence_proxy_async_smem();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot, t_s = tmem_base, t_o = tmem_base + 128;

  if (warp == 0) {
    if (lane == 0) {
      const int* table = p.block_tables + (size_t)seq * p.max_blocks;
      const int last = (kv_len - 1) / kPage * kPage;                 // pages past the sequence repeat its last one (finite values)
      for (int it = 0; it < n_tiles; ++it) {
        const int b = it & 1;
        int rows[kTile / kPage];
#pragma unroll
        for (int pg = 0; pg < kTile / kPage; ++pg) rows[pg] = page_row(p, table, min(it * kTile + pg * kPage, last), kvh);
        if (it >= 2 && !mbar_wait(&k_empty[b], ((it >> 1) - 1) & 1, abort_flag)) break;
        mbar_expect_tx(&k_full[b], TB + kTile * 4);
#pragma unroll
        for (int pg = 0; pg < kTile / kPage; ++pg) {
#pragma unroll
          for (int h = 0; h < D / 64; ++h) tma_load_2d(sk + b * TB + h * kHalf + pg * (kPage * 128), &tma_k, &k_full[b], 64 * h, rows[pg]);
          bulk_load(skf + b * kTile + pg * kPage, p.key_factor + rows[pg], kPage * 4, &k_full[b]);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(128, 128, 1, 1);
      constexpr uint32_t idesc_pv = make_idesc(128, D, 1, 1) | (1u << 16);      // B is MN-major
      const uint32_t q_addr = smem_u32(sq), k_addr = smem_u32(sk);
      for (int it = 0; it < n_tiles; ++it) {
        const uint32_t kb = k_addr + (it & 1) * TB;
        if (!mbar_wait(&k_full[it & 1], (it >> 1) & 1, abort_flag)) break;
        tc_fence_after_sync();
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
          const uint32_t off = (k >> 2) * kHalf + (k & 3) * 32;
          tc_mma_bf16(t_s, make_smem_desc_sw128(q_addr + off), make_smem_desc_sw128(kb + off), idesc_s, k > 0);
        }
        tc_commit(s_full);
        if (!mbar_wait(p_ready, it & 1, abort_flag)) break;
        tc_fence_after_sync();
#pragma unroll
        for (int k = 0; k < kTile / 16; ++k) {
          const uint32_t a = t_s + 32 * (k >> 1) + 8 * (k & 1);
          const uint64_t v = desc_mn_major<D>(kb + k * 2048);
          tc_mma_bf16_ts(t_o, a, v, idesc_pv, it > 0 || k > 0);
          tc_mma_bf16_ts(t_o, a + 16, v, idesc_pv, 1);
        }
        tc_commit(&k_empty[it & 1]);
        if (it == n_tiles - 1) tc_commit(o_done);
      }
    }
  } else {
    const int r = (warp & 3) * 32 + lane;                            // the lane quarter this warp may touch
    const uint32_t lane_off = (uint32_t)((warp & 3) * 32) << 16;
    const bool valid = r < n_rows;
    const int tok = q0 + (row0 + r) / p.group, head = kvh * p.group + (row0 + r) % p.group;
    const int lim = valid ? first_pos + (row0 + r) / p.group + 1 : 0;
    const float rf = valid ? row_factor<CAP>(p, tok, head) : 0.f, cap2 = p.softcap * kLog2e;
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int it = 0; it < n_tiles; ++it) {
      const int tok0 = it * kTile;
      // the factors arrived with the tile (this wait is over before the scores' one)
      if (!mbar_wait(&k_full[it & 1], (it >> 1) & 1, abort_flag) || !mbar_wait(s_full, it & 1, abort_flag)) { ok = false; break; }
      tc_fence_after_sync();
      const float* kf = skf + (it & 1) * kTile;
      if (tok0 + kTile <= lim_first && n_rows == kRows)              // every row of the CTA sees the whole tile
        softmax_tile<D, true, CAP, FIXED>(t_s + lane_off, t_o + lane_off, kf, rf, cap2, 0, it > 0, m_used, l);
      else
        softmax_tile<D, false, CAP, FIXED>(t_s + lane_off, t_o + lane_off, kf, rf, cap2, lim - tok0, it > 0, m_used, l);
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    if (ok && mbar_wait(o_done, 0, abort_flag)) {
      tc_fence_after_sync();
      const float inv = l > 0.f ? 1.f / l : 0.f;
      bf16* dst = p.out + (long long)tok * p.ldo + (long long)head * p.dim;
#pragma unroll 1
      for (int cc = 0; cc < D / 32; ++cc) {
        uint32_t o[32];
        tmem_ld_32x32(t_o + lane_off + 32 * cc, o);
        tmem_ld_wait();
        if (!valid) continue;
        if (p.vec) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (32 * cc + i >= p.dim) continue;
            uint4 w;
            w.x = pack_bf16x2(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv);
            w.y = pack_bf16x2(__uint_as_float(o[i + 2]) * inv, __uint_as_float(o[i + 3]) * inv);
            w.z = pack_bf16x2(__uint_as_float(o[i + 4]) * inv, __uint_as_float(o[i + 5]) * inv);
            w.w = pack_bf16x2(__uint_as_float(o[i + 6]) * inv, __uint_as_float(o[i + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + 32 * cc + i) = w;
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (32 * cc + i < p.dim) dst[32 * cc + i] = __float2bfloat16(__uint_as_float(o[i]) * inv);
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) { tc_fence_after_sync(); tmem_dealloc(tmem_base, 256); }
  if (threadIdx.x == 0 && *abort_flag && p.status) atomicCAS(p.status, FLLM_OK, FLLM_ERR_MBAR_TIMEOUT);
}

// ------------------------------------------------------------------------------------------ host
const CUtensorMap& key_map(const void* cache, uint64_t rows, int D) {
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
  const Key key{cache, rows, D};
  auto it = maps.find(key);
  if (it == maps.end()) {
    if (maps.size() > 4096) maps.clear();
    it = maps.emplace(key, make_tmap_2d(cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, rows, D, D * 2, kPage, 64, true)).first;
  }
  return it->second;
}

// key slices of a step whose sequences all run in the decode kernel
int decode_splits(int num_seqs, int max_q_len, int H, int G, int max_kv_len) {
  const long long ctas = (long long)num_seqs * G * ((max_q_len * (H / G) + 15) / 16);
  const int pages = (max_kv_len + kPage - 1) / kPage;
  if (ctas >= sm_count()) return 1;
  return std::max(1, (int)std::min<long long>({(2 * sm_count() + ctas - 1) / ctas, (pages + 7) / 8, 32}));
}

template <int D, bool CAP, bool FIXED>
int launch_tc(Tied a, const TiedAttnParams& p, int splits, cudaStream_t s) {
  static bool configured[kMaxDevices] = {};
  if (first_call_on_device(configured)) {
    cuda_check(cudaFuncSetAttribute(tied_decode_kernel<D, CAP, FIXED>, cudaFuncAttributeMaxDynamicSharedMemorySize, DecodeTile<D>::kTotal), "tied_decode smem");
    cuda_check(cudaFuncSetAttribute(tied_prefill_kernel<D, CAP, FIXED>, cudaFuncAttributeMaxDynamicSharedMemorySize, prefill_smem<D>()), "tied_prefill smem");
  }
  int launches = 0;
  const int max_rows = p.max_q_len * a.group;
  if (p.min_q_len * a.group <= kDecodeRows) {
    a.splits = max_rows <= kDecodeRows ? splits : 1;      // partial results of longer sequences do not exist
    const int row_tiles = (std::min(max_rows, kDecodeRows) + 15) / 16;
    launch_pdl(tied_decode_kernel<D, CAP, FIXED>, dim3(a.G * row_tiles, p.num_seqs, a.splits), dim3(128), DecodeTile<D>::kTotal, s, a, row_tiles, (int)kDecodeRows);
    ++launches;
    if (a.splits > 1) {
      launch_pdl(tied_merge_kernel<D>, dim3((p.tokens * a.H + 3) / 4), dim3(128), 0, s, a, p.tokens);
      ++launches;
    }
  }
  if (max_rows > kDecodeRows) {
    const CUtensorMap& map = key_map(p.cache, (uint64_t)p.num_blocks * a.G * a.block_size, D);
    tied_prefill_kernel<D, CAP, FIXED><<<dim3((max_rows + kRows - 1) / kRows, a.G, p.num_seqs), kThreads, prefill_smem<D>(), s>>>(map, a, kDecodeRows + 1);
    ++launches;
  }
  cuda_check(cudaGetLastError(), "attention_tied launch");
  return launches;
}

template <typename T>
void launch_simple(const TiedAttnParams& p, cudaStream_t s) {
  constexpr int NW = 4;
  const size_t smem = (size_t)(p.dim + NW * p.dim + 2 * NW) * sizeof(float);
  const dim3 grid(p.H, p.tokens);
  if (p.dim <= 64) tied_simple_kernel<T, 2, NW><<<grid, NW * 32, smem, s>>>(p);
  else if (p.dim <= 128) tied_simple_kernel<T, 4, NW><<<grid, NW * 32, smem, s>>>(p);
  else if (p.dim <= 256) tied_simple_kernel<T, 8, NW><<<grid, NW * 32, smem, s>>>(p);
  else if (p.dim <= 512) tied_simple_kernel<T, 16, NW><<<grid, NW * 32, smem, s>>>(p);
  else throw std::runtime_error("attention_tied: heads of at most 512 values");
  cuda_check(cudaGetLastError(), "tied_simple_kernel");
}
}  // namespace

bool attention_tied_tc_supported(int W, int block_size, int f32) { return !f32 && (W == 64 || W == 128) && block_size % kPage == 0; }

// key slices the tensor-core path uses for a step (1: no workspace needed)
int attention_tied_splits(int num_seqs, int max_q_len, int H, int G, int max_kv_len) {
  return max_q_len * (H / G) <= kDecodeRows ? decode_splits(num_seqs, max_q_len, H, G, max_kv_len) : 1;
}
size_t attention_tied_workspace_bytes(int tokens, int H, int W, int splits) {
  return splits > 1 ? (size_t)tokens * H * splits * (W + 2) * sizeof(float) : 0;
}

int attention_tied(const TiedAttnParams& p, int splits, void* workspace, size_t workspace_bytes, bool tensor_cores, int* status, cudaStream_t s) {
  if (p.tokens <= 0) return 0;
  if (p.tokens > 65535 || p.num_seqs > 65535) throw std::runtime_error("attention_tied: at most 65535 rows and sequences in a step");
  if (!tensor_cores || !attention_tied_tc_supported(p.W, p.block_size, p.f32)) {
    if (p.f32) launch_simple<float>(p, s);
    else launch_simple<bf16>(p, s);
    return 1;
  }
  splits = std::max(splits, 1);
  if (workspace_bytes < attention_tied_workspace_bytes(p.tokens, p.H, p.W, splits))
    throw std::runtime_error("attention_tied: workspace too small for the requested key slices");
  Tied a{};
  a.q = static_cast<const bf16*>(p.q), a.ldq = p.ldq, a.q_factor = p.q_factor, a.cache = static_cast<const bf16*>(p.cache), a.key_factor = p.key_factor;
  a.block_tables = p.block_tables, a.max_blocks = p.max_blocks, a.q_starts = p.q_starts, a.positions = p.positions;
  a.out = static_cast<bf16*>(p.out), a.ldo = p.ldo;
  a.H = p.H, a.G = p.G, a.group = p.H / p.G, a.dim = p.dim, a.block_size = p.block_size, a.softcap = p.softcap;
  a.vec = p.dim % 8 == 0 && p.ldq % 8 == 0 && p.ldo % 8 == 0 && ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.out)) & 15) == 0;
  a.ws_o = static_cast<float*>(workspace);
  a.ws_ml = a.ws_o != nullptr ? a.ws_o + (size_t)p.tokens * p.H * splits * p.W : nullptr;
  a.status = status;
  const bool cap = p.softcap > 0.f, fixed = cap && p.softcap <= kFixedCap;
#define FLLM_TIED(D_)                                                             \
  return fixed ? launch_tc<D_, true, true>(a, p, splits, s)                       \
               : (cap ? launch_tc<D_, true, false>(a, p, splits, s) : launch_tc<D_, false, false>(a, p, splits, s));
  if (p.W == 64) { FLLM_TIED(64) }
  FLLM_TIED(128)
#undef FLLM_TIED
}

void tied_prepare(const TiedPrepareParams& params, cudaStream_t s) {
  if (params.tokens <= 0) return;
  TiedPrepareParams p = params;
  const uintptr_t any = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.cache) | reinterpret_cast<uintptr_t>(p.q_out);
  p.vec = p.dim % 4 == 0 && p.k_offset % 4 == 0 && p.W % 4 == 0 && any % 16 == 0 &&
          (p.partials ? p.width % 4 == 0 && p.plane % 4 == 0 && p.ld_qout % 4 == 0 && reinterpret_cast<uintptr_t>(p.partials) % 16 == 0 : p.ldx % 4 == 0);
  const unsigned blocks = (unsigned)(((long long)p.tokens * (p.H + p.G) + 3) / 4);
  if (p.f32) launch_pdl(tied_prepare_kernel<float>, dim3(blocks), dim3(128), 0, s, p);
  else launch_pdl(tied_prepare_kernel<bf16>, dim3(blocks), dim3(128), 0, s, p);
  cuda_check(cudaGetLastError(), "tied_prepare_kernel");
}

}  // namespace fllm
