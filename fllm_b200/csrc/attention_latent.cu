// Latent attention for any sizes: a token's cache row is [latent (R) | rotated shared key part (dr) | zeros] padded to a
// multiple of 16 values (W), every head is one query of that layout (the key up-projection is absorbed into it), and a
// head's output is the weighted sum of the latents (the value up-projection follows). attention_mla.cu holds the kernels
// for the one width of the DeepSeek family; the ones here take R, dr and the head count as arguments, put the rows of
// neighbouring tokens beside the heads of one token, and exist in bf16 and in fp32.
//
// Rows of one sequence are numbered token * H + head, so a tile of 16 * MT consecutive rows shares each key tile: with few
// heads a prompt fills the tile with tokens, with many heads one decoded token does. Weights are kept in fp32; for the
// tensor-core product with the latents a weight travels as the sum of two bf16 values (16 significant bits).
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>
#include <stdexcept>

#include "fllm_ops.h"
#include "ptx.cuh"
#include "tma_host.h"

namespace fllm {
namespace {
using bf16 = __nv_bfloat16;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16(v); }

// ------------------------------------------------------------------------------------------ cache rows and rotated queries
// One CTA per token: RMS norm of the latent and rotation of the shared key part into the token's cache row (skipped when
// `ckv` is null, the layer reads another layer's rows, and for padding rows, slot < 0); rotation of every head's rotary
// part into columns [R, R + dr) of its query row q_out[h][t], zeros behind. style 0 turns the pairs (i, i + dr / 2), style 1
// neighbours (2 i, 2 i + 1).
template <typename T>
__global__ void __launch_bounds__(128) latent_prepare_kernel(const LatentPrepareParams p) {
  const int t = blockIdx.x, tid = threadIdx.x;
  const float pos = (float)p.positions[t];
  const int half = p.dr / 2;
  const T* q = static_cast<const T*>(p.q) + (long long)t * p.ld_q + p.q_rope_offset;
  T* qo = static_cast<T*>(p.q_out) + (long long)t * p.W + p.R;
  for (int i = tid; i < p.H * half; i += 128) {
    const int h = i / half, f = i % half;
    float sn, cs;
    sincosf(pos * p.inv_freq[f], &sn, &cs);
    sn *= p.attn_factor, cs *= p.attn_factor;
    const int a = p.style ? 2 * f : f, b = p.style ? 2 * f + 1 : f + half;
    const T* src = q + (long long)h * p.q_head;
    const float u = to_f32(src[a]), v = to_f32(src[b]);
    T* dst = qo + (long long)h * p.q_out_h;
    dst[a] = from_f32<T>(u * cs - v * sn);
    dst[b] = from_f32<T>(v * cs + u * sn);
  }
  const int tail = p.W - p.R - p.dr;
  for (int i = tid; i < p.H * tail; i += 128) qo[(long long)(i / tail) * p.q_out_h + p.dr + i % tail] = from_f32<T>(0.f);
  if (p.ckv == nullptr) return;
  const int slot = p.slots[t];
  if (slot < 0) return;
  const T* row = static_cast<const T*>(p.ckv) + (long long)t * p.ld_ckv;
  const T* w = static_cast<const T*>(p.norm_w);
  T* dst = static_cast<T*>(p.cache) + (long long)slot * p.W;
  __shared__ float red[4];
  float ss = 0.f;
  for (int i = tid; i < p.R; i += 128) {
    const float v = to_f32(row[i]);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  const float inv = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)p.R + p.eps);
  for (int i = tid; i < p.R; i += 128) dst[i] = from_f32<T>(to_f32(row[i]) * inv * to_f32(w[i]));
  for (int f = tid; f < half; f += 128) {
    float sn, cs;
    sincosf(pos * p.inv_freq[f], &sn, &cs);
    sn *= p.attn_factor, cs *= p.attn_factor;
    const int a = p.style ? 2 * f : f, b = p.style ? 2 * f + 1 : f + half;
    const float u = to_f32(row[p.R + a]), v = to_f32(row[p.R + b]);
    dst[p.R + a] = from_f32<T>(u * cs - v * sn);
    dst[p.R + b] = from_f32<T>(v * cs + u * sn);
  }
  for (int i = tid; i < tail; i += 128) dst[p.R + p.dr + i] = from_f32<T>(0.f);
}

// out[t][h * dv + j] = o[h][t][j] * sigmoid(gate[t][h]); columns beyond H * dv are zero
template <typename T>
__global__ void __launch_bounds__(256) head_gate_kernel(const T* __restrict__ o, long long o_h, long long o_t, const T* __restrict__ gate,
                                                        long long ld_gate, T* __restrict__ out, long long ld_out, int H, int dv, int cols) {
  const int t = blockIdx.x;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) {
    float v = 0.f;
    if (c < H * dv) {
      const int h = c / dv;
      v = to_f32(o[h * o_h + t * o_t + c - h * dv]);
      if (gate != nullptr) v *= 1.f / (1.f + expf(-to_f32(gate[t * ld_gate + h])));
    }
    out[t * ld_out + c] = from_f32<T>(v);
  }
}

// ------------------------------------------------------------------------------------------ CUDA-core attention
// One CTA per (token, head); its warps take every NW-th key with an online softmax each and are merged through shared
// memory. Lane l owns the columns l, l + 32, ... Any W; R up to 32 * EV.
template <typename T, int EV, int NW>
__global__ void __launch_bounds__(NW * 32) latent_simple_kernel(const LatentAttnParams p) {
  extern __shared__ float sm[];
  float* sq = sm;                              // [W] query row * scale
  float* sacc = sq + p.W;                      // [NW][R]
  float* sml = sacc + NW * p.R;                // [NW][2] maximum and sum
  const int h = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* q = static_cast<const T*>(p.q) + (long long)h * p.q_h + (long long)t * p.W;
  const T* cache = static_cast<const T*>(p.cache);
  for (int i = threadIdx.x; i < p.W; i += NW * 32) sq[i] = to_f32(q[i]) * p.scale;
  __syncthreads();
  const int kv_len = p.positions[t] + 1;
  const int* table = p.block_tables + (size_t)p.row_seq[t] * p.max_blocks;
  float m = -INFINITY, l = 0.f, acc[EV];
#pragma unroll
  for (int e = 0; e < EV; ++e) acc[e] = 0.f;
  for (int j = warp; j < kv_len; j += NW) {
    const T* row = cache + ((size_t)table[j / p.block_size] * p.block_size + j % p.block_size) * p.W;
    float s = 0.f, v[EV];
#pragma unroll
    for (int e = 0; e < EV; ++e) {
      const int c = lane + 32 * e;
      v[e] = c < p.R ? to_f32(row[c]) : 0.f;
      if (c < p.R) s = fmaf(v[e], sq[c], s);
    }
    for (int c = p.R + lane; c < p.W; c += 32) s = fmaf(to_f32(row[c]), sq[c], s);
    s = warp_sum(s);
    const float mn = fmaxf(m, s), corr = expf(m - mn), pr = expf(s - mn);
    l = l * corr + pr;
#pragma unroll
    for (int e = 0; e < EV; ++e) acc[e] = fmaf(acc[e], corr, pr * v[e]);
    m = mn;
  }
#pragma unroll
  for (int e = 0; e < EV; ++e)
    if (lane + 32 * e < p.R) sacc[warp * p.R + lane + 32 * e] = acc[e];
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
  T* out = static_cast<T*>(p.out) + (long long)h * p.o_h + (long long)t * p.o_t;
  for (int i = threadIdx.x; i < p.R; i += NW * 32) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) v = fmaf(sacc[w * p.R + i], c[w], v);
    out[i] = from_f32<T>(v / tot);
  }
}

// ------------------------------------------------------------------------------------------ tensor-core attention (bf16)
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
__device__ __forceinline__ void ldsm_x2(uint32_t& r0, uint32_t& r1, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(smem_u32(p)));
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

constexpr int kWarps = 8;

template <int MT, int KT>
struct LatentTile {
  static constexpr int ROWS = 16 * MT;
  static constexpr int WPM = kWarps / MT;                 // warps that share the keys of one 16-row tile
  static constexpr int NPW = KT / 8 / WPM;                // 8-key groups of a warp in the score phase
  static constexpr int PP = KT + 8;                       // pitch of a weight row
  // pitches are odd multiples of 16 bytes, so the eight rows of an ldmatrix fetch fall into distinct banks
  static size_t smem_bytes(int W) {
    return (size_t)(ROWS + 2 * KT) * (W + 8) * 2 + (size_t)2 * ROWS * PP * 2 + (size_t)2 * WPM * ROWS * 4;
  }
};

// Grid (row tiles of a sequence, sequences, key slices). Per key tile (double-buffered cp.async): warp w computes the scores
// of its 16-row tile for NPW groups of 8 keys, the row maxima meet in shared memory, weights go to shared memory as two
// bf16 terms, and every warp accumulates all rows for its NTW groups of 8 latent columns. With several key slices a CTA
// leaves (maximum, sum, unnormalised output) in the workspace for latent_merge_kernel.
template <int MT, int KT, int NTW>
__global__ void __launch_bounds__(kWarps * 32) latent_tc_kernel(const LatentAttnParams p, float scale_log2, int splits,
                                                                float* __restrict__ part_o, float* __restrict__ part_ml) {
  using L = LatentTile<MT, KT>;
  constexpr int ROWS = L::ROWS, WPM = L::WPM, NPW = L::NPW, PP = L::PP;
  extern __shared__ __align__(128) unsigned char smem_raw[];
  const int pitch = p.W + 8;
  bf16* sq = reinterpret_cast<bf16*>(smem_raw);
  bf16* sk = sq + ROWS * pitch;
  bf16* sph = sk + 2 * KT * pitch;
  bf16* spl = sph + ROWS * PP;
  float* smax = reinterpret_cast<float*>(spl + ROWS * PP);      // [WPM][ROWS]
  float* ssum = smax + WPM * ROWS;                              // [WPM][ROWS]

  const int seq = blockIdx.y, split = blockIdx.z;
  const int t0 = p.q_starts[seq], n_rows = (p.q_starts[seq + 1] - t0) * p.H;
  const int row0 = blockIdx.x * ROWS;
  if (row0 >= n_rows) return;
  const int rows = min(ROWS, n_rows - row0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, tq = lane & 3, j4 = lane >> 3;
  const int* table = p.block_tables + (size_t)p.row_seq[t0 + row0 / p.H] * p.max_blocks;
  const int kv_max = p.positions[t0 + (row0 + rows - 1) / p.H] + 1;
  const int tiles = (kv_max + KT - 1) / KT;
  const int per = (tiles + splits - 1) / splits;
  const int tile_lo = split * per, tile_hi = min(tiles, tile_lo + per);
  const bf16* qg = static_cast<const bf16*>(p.q);
  const bf16* cache = static_cast<const bf16*>(p.cache);
  const int cpr = p.W / 8;                                      // 16-byte chunks of a row

  for (int i = tid; i < ROWS * cpr; i += kWarps * 32) {
    const int r = i / cpr, c = i - r * cpr;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < rows) {
      const int t = t0 + (row0 + r) / p.H, h = (row0 + r) % p.H;
      v = *reinterpret_cast<const uint4*>(qg + (long long)h * p.q_h + (long long)t * p.W + c * 8);
    }
    *reinterpret_cast<uint4*>(sq + r * pitch + c * 8) = v;
  }
  constexpr int KPW = KT / kWarps;                              // key rows a warp brings in
  auto load_tile = [&](int tile, int buf) {
    const int key0 = tile * KT + warp * KPW;
    const bf16* mine = nullptr;
    if (lane < KPW && key0 + lane < kv_max) {
      const int key = key0 + lane;
      mine = cache + ((size_t)table[key / p.block_size] * p.block_size + key % p.block_size) * p.W;
    }
#pragma unroll
    for (int r = 0; r < KPW; ++r) {
      const bf16* src = reinterpret_cast<const bf16*>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(mine), r));
      bf16* dst = sk + (buf * KT + warp * KPW + r) * pitch;
      for (int c = lane; c < cpr; c += 32) {
        if (src != nullptr) cp_async16(dst + c * 8, src + c * 8);
        else *reinterpret_cast<uint4*>(dst + c * 8) = make_uint4(0, 0, 0, 0);     // keys past the end must not feed NaNs into the product
      }
    }
  };

  // visible length of the lane's two rows in every 16-row tile (0 for rows past the end: all masked)
  int vis[MT][2];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = mt * 16 + g + 8 * i;
      vis[mt][i] = r < rows ? p.positions[t0 + (row0 + r) / p.H] + 1 : 0;
    }
  float o[MT][NTW][4];
  float m[MT][2], l[2] = {0.f, 0.f};
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
    m[mt][0] = m[mt][1] = -INFINITY;
#pragma unroll
    for (int i = 0; i < NTW; ++i) o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f;
  }
  const int wm = warp / WPM, wn = warp % WPM;                   // 16-row tile and key share of this warp in the score phase
  const int ksteps = p.W / 16;

  if (tile_lo < tile_hi) load_tile(tile_lo, 0);
  cp_async_commit();
  for (int tile = tile_lo; tile < tile_hi; ++tile) {
    const int buf = (tile - tile_lo) & 1;
    if (tile + 1 < tile_hi) load_tile(tile + 1, buf ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const bf16* kt = sk + buf * KT * pitch;
    // ---- scores of 16 rows x NPW * 8 keys
    float s[NPW][4];
#pragma unroll
    for (int n = 0; n < NPW; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
    const bf16* qw = sq + (wm * 16 + (lane & 15)) * pitch + (lane >> 4) * 8;
    if constexpr (NPW == 1) {
      float s2[4] = {0.f, 0.f, 0.f, 0.f};                       // two chains
      const bf16* kw = kt + (wn * 8 + (lane & 7)) * pitch;
      int kk = 0;
      for (; kk + 1 < ksteps; kk += 2) {
        uint32_t a0[4], a1[4], b[4];
        ldsm_x4(a0, qw + kk * 16);
        ldsm_x4(a1, qw + kk * 16 + 16);
        ldsm_x4(b, kw + kk * 16 + j4 * 8);
        mma_bf16(s[0], a0, b[0], b[1]);
        mma_bf16(s2, a1, b[2], b[3]);
      }
      if (kk < ksteps) {
        uint32_t a0[4], b0, b1;
        ldsm_x4(a0, qw + kk * 16);
        ldsm_x2(b0, b1, kw + kk * 16 + (j4 & 1) * 8);
        mma_bf16(s[0], a0, b0, b1);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) s[0][e] += s2[e];
    } else {
      const bf16* kw = kt + (wn * NPW * 8 + (j4 >> 1) * 8 + (lane & 7)) * pitch + (j4 & 1) * 8;
#pragma unroll 2
      for (int kk = 0; kk < ksteps; ++kk) {
        uint32_t a[4];
        ldsm_x4(a, qw + kk * 16);
#pragma unroll
        for (int n = 0; n + 1 < NPW; n += 2) {
          uint32_t b[4];
          ldsm_x4(b, kw + n * 8 * pitch + kk * 16);
          mma_bf16(s[n], a, b[0], b[1]);
          mma_bf16(s[n + 1], a, b[2], b[3]);
        }
      }
    }
    int v0 = 0, v1 = 0;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
      if (mt == wm) v0 = vis[mt][0], v1 = vis[mt][1];
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int n = 0; n < NPW; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = tile * KT + (wn * NPW + n) * 8 + 2 * tq + (e & 1);
        const float v = key < (e < 2 ? v0 : v1) ? s[n][e] * scale_log2 : -INFINITY;
        s[n][e] = v;
        if (e < 2) mx0 = fmaxf(mx0, v);
        else mx1 = fmaxf(mx1, v);
      }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    if (tq == 0) smax[wn * ROWS + wm * 16 + g] = mx0, smax[wn * ROWS + wm * 16 + g + 8] = mx1;
    __syncthreads();
    // ---- new maxima of all rows (every warp rescales its columns of every row), weights of this warp's rows
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      float mn[2], c[2], base[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mn[i] = m[mt][i];
#pragma unroll
        for (int w = 0; w < WPM; ++w) mn[i] = fmaxf(mn[i], smax[w * ROWS + mt * 16 + g + 8 * i]);
        base[i] = mn[i] == -INFINITY ? 0.f : mn[i];             // nothing visible yet: all weights stay zero
        c[i] = exp2f(m[mt][i] - base[i]);
        m[mt][i] = mn[i];
      }
#pragma unroll
      for (int n = 0; n < NTW; ++n) o[mt][n][0] *= c[0], o[mt][n][1] *= c[0], o[mt][n][2] *= c[1], o[mt][n][3] *= c[1];
      if (mt == wm) {
        l[0] *= c[0], l[1] *= c[1];
#pragma unroll
        for (int n = 0; n < NPW; ++n) {
          const int col = (wn * NPW + n) * 8 + 2 * tq;
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float p0 = exp2f(s[n][2 * i] - base[i]), p1 = exp2f(s[n][2 * i + 1] - base[i]);
            l[i] += p0 + p1;
            const uint32_t hi = pack_bf16x2(p0, p1);
            const float2 back = unpack_bf16x2(hi);
            const int at = (mt * 16 + g + 8 * i) * PP + col;
            *reinterpret_cast<uint32_t*>(sph + at) = hi;
            *reinterpret_cast<uint32_t*>(spl + at) = pack_bf16x2(p0 - back.x, p1 - back.y);
          }
        }
      }
    }
    __syncthreads();
    // ---- O += P V over this warp's columns (16 at a time; columns past the latent are skipped)
#pragma unroll
    for (int kq = 0; kq < KT / 16; ++kq) {
      uint32_t vb[NTW / 2][4];
#pragma unroll
      for (int n = 0; n < NTW / 2; ++n) {
        const int col = (warp * (NTW / 2) + n) * 16;
        if (col < p.R) ldsm_x4_t(vb[n], kt + (kq * 16 + (j4 & 1) * 8 + (lane & 7)) * pitch + col + (j4 >> 1) * 8);
      }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t ph[4], pl[4];
        ldsm_x4(ph, sph + (mt * 16 + (lane & 15)) * PP + kq * 16 + (lane >> 4) * 8);
        ldsm_x4(pl, spl + (mt * 16 + (lane & 15)) * PP + kq * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int n = 0; n < NTW / 2; ++n) {
          if ((warp * (NTW / 2) + n) * 16 >= p.R) continue;
          mma_bf16(o[mt][2 * n], ph, vb[n][0], vb[n][1]);
          mma_bf16(o[mt][2 * n + 1], ph, vb[n][2], vb[n][3]);
          mma_bf16(o[mt][2 * n], pl, vb[n][0], vb[n][1]);
          mma_bf16(o[mt][2 * n + 1], pl, vb[n][2], vb[n][3]);
        }
      }
    }
    __syncthreads();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    if (tq == 0) ssum[wn * ROWS + wm * 16 + g + 8 * i] = l[i];
  }
  __syncthreads();
  bf16* out = static_cast<bf16*>(p.out);
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = mt * 16 + g + 8 * i;
      if (r >= rows) continue;
      float tot = 0.f;
#pragma unroll
      for (int w = 0; w < WPM; ++w) tot += ssum[w * ROWS + r];
      const int t = t0 + (row0 + r) / p.H, h = (row0 + r) % p.H;
      const size_t pr = ((size_t)t * p.H + h) * splits + split;
      if (splits > 1 && warp == 0 && tq == 0) part_ml[2 * pr] = m[mt][i], part_ml[2 * pr + 1] = tot;
      const float inv = tot > 0.f ? 1.f / tot : 0.f;
#pragma unroll
      for (int n = 0; n < NTW; ++n) {
        const int col = (warp * NTW + n) * 8 + 2 * tq;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (col + e >= p.R) continue;
          if (splits > 1) part_o[pr * p.R + col + e] = o[mt][n][2 * i + e];
          else out[(long long)h * p.o_h + (long long)t * p.o_t + col + e] = __float2bfloat16(o[mt][n][2 * i + e] * inv);
        }
      }
    }
}

// out(t, h) = sum_s exp2(m_s - m) O_s / sum_s exp2(m_s - m) l_s
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits,
                                                           const LatentAttnParams p) {
  const int h = blockIdx.x, t = blockIdx.y;
  const size_t r = ((size_t)t * p.H + h) * splits;
  float mm = -INFINITY;
  for (int s = 0; s < splits; ++s) mm = fmaxf(mm, part_ml[2 * (r + s)]);
  float tot = 0.f;
  for (int s = 0; s < splits; ++s)
    if (part_ml[2 * (r + s)] != -INFINITY) tot = fmaf(part_ml[2 * (r + s) + 1], exp2f(part_ml[2 * (r + s)] - mm), tot);
  const float inv = tot > 0.f ? 1.f / tot : 0.f;
  bf16* out = static_cast<bf16*>(p.out) + (long long)h * p.o_h + (long long)t * p.o_t;
  for (int c = threadIdx.x; c < p.R; c += 128) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = part_ml[2 * (r + s)];
      if (ms != -INFINITY) v = fmaf(part_o[(r + s) * p.R + c], exp2f(ms - mm), v);
    }
    out[c] = __float2bfloat16(v * inv);
  }
}

template <int MT, int KT, int NTW>
void launch_tc(const LatentAttnParams& p, int splits, float* po, float* pml, cudaStream_t s) {
  using L = LatentTile<MT, KT>;
  static bool configured = false;
  if (!configured) {
    cuda_check(cudaFuncSetAttribute(latent_tc_kernel<MT, KT, NTW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024), "latent_tc_kernel");
    configured = true;
  }
  const int tiles = (p.max_q_len * p.H + L::ROWS - 1) / L::ROWS;
  latent_tc_kernel<MT, KT, NTW><<<dim3(tiles, p.num_seqs, splits), kWarps * 32, L::smem_bytes(p.W), s>>>(p, p.scale * kLog2e, splits, po, pml);
  cuda_check(cudaGetLastError(), "latent_tc_kernel");
}

template <typename T, int NW>
void launch_simple(const LatentAttnParams& p, cudaStream_t s) {
  const size_t smem = (size_t)(p.W + NW * p.R + 2 * NW) * sizeof(float);
  const dim3 grid(p.H, p.tokens);
  auto go = [&](auto kernel) {
    if (smem > 48 * 1024) cuda_check(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024), "latent_simple_kernel");
    kernel<<<grid, NW * 32, smem, s>>>(p);
  };
  if (p.R <= 64) go(latent_simple_kernel<T, 2, NW>);
  else if (p.R <= 128) go(latent_simple_kernel<T, 4, NW>);
  else if (p.R <= 256) go(latent_simple_kernel<T, 8, NW>);
  else if (p.R <= 512) go(latent_simple_kernel<T, 16, NW>);
  else if (p.R <= 1024) go(latent_simple_kernel<T, 32, NW>);
  else throw std::runtime_error("attention_latent: latents of at most 1024 values");
  cuda_check(cudaGetLastError(), "latent_simple_kernel");
}

int tiles_m(int max_rows) { return max_rows <= 16 ? 1 : (max_rows <= 32 ? 2 : 4); }
}  // namespace

// Whether the tensor-core kernel takes this layout (bf16): the latent fits its columns and the tile its shared memory.
bool attention_latent_tc_supported(int W, int R, int max_rows) {
  if (R > 512 || (W & 15)) return false;
  const int mt = tiles_m(max_rows);
  const size_t need = mt == 1 ? LatentTile<1, 64>::smem_bytes(W) : mt == 2 ? LatentTile<2, 64>::smem_bytes(W) : LatentTile<4, 32>::smem_bytes(W);
  return need <= 227 * 1024;
}

// Key slices of a step: enough CTAs for the machine, a few key tiles per slice.
int attention_latent_splits(int num_seqs, int tokens, int max_q_len, int H, int max_kv_len) {
  const int mt = tiles_m(max_q_len * H);
  const long long ctas = std::max((long long)num_seqs, ((long long)tokens * H + 16 * mt - 1) / (16 * mt));
  const int tiles = (max_kv_len + 63) / 64;
  int splits = 1;
  while (splits < 16 && ctas * splits < 148 && tiles / (splits * 2) >= 4) splits *= 2;
  return splits;
}

size_t attention_latent_workspace_bytes(int tokens, int H, int R, int splits) {
  return splits > 1 ? (size_t)tokens * H * splits * (R + 2) * sizeof(float) : 0;
}

int attention_latent(const LatentAttnParams& p, int splits, void* workspace, size_t workspace_bytes, bool tensor_cores, cudaStream_t s) {
  if (p.tokens <= 0) return 0;
  if (p.tokens > 65535 || p.num_seqs > 65535) throw std::runtime_error("attention_latent: at most 65535 rows and sequences in a step");
  if (p.f32) {
    launch_simple<float, 4>(p, s);
    return 1;
  }
  const bool aligned = ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.cache)) & 15) == 0 && (p.q_h & 7) == 0;
  if (!tensor_cores || !aligned || !attention_latent_tc_supported(p.W, p.R, p.max_q_len * p.H)) {
    launch_simple<bf16, 4>(p, s);
    return 1;
  }
  if (splits < 1) splits = 1;
  if (workspace_bytes < attention_latent_workspace_bytes(p.tokens, p.H, p.R, splits))
    throw std::runtime_error("attention_latent: workspace too small for the requested key slices");
  float* po = static_cast<float*>(workspace);
  float* pml = po != nullptr ? po + (size_t)p.tokens * p.H * splits * p.R : nullptr;
  const int mt = tiles_m(p.max_q_len * p.H), ntw = p.R <= 128 ? 2 : (p.R <= 256 ? 4 : 8);
#define FLLM_LAT(MT_, KT_)                                                   \
  if (ntw == 2) launch_tc<MT_, KT_, 2>(p, splits, po, pml, s);               \
  else if (ntw == 4) launch_tc<MT_, KT_, 4>(p, splits, po, pml, s);          \
  else launch_tc<MT_, KT_, 8>(p, splits, po, pml, s);
  if (mt == 1) { FLLM_LAT(1, 64) }
  else if (mt == 2) { FLLM_LAT(2, 64) }
  else { FLLM_LAT(4, 32) }
#undef FLLM_LAT
  if (splits > 1) {
    latent_merge_kernel<<<dim3(p.H, p.tokens), 128, 0, s>>>(po, pml, splits, p);
    cuda_check(cudaGetLastError(), "latent_merge_kernel");
    return 2;
  }
  return 1;
}

void latent_prepare(const LatentPrepareParams& p, cudaStream_t s) {
  if (p.tokens <= 0) return;
  if (p.dr & 1 || p.R + p.dr > p.W) throw std::runtime_error("latent_prepare: an even rotary width, rows of at least latent + rotary values");
  if (p.f32) latent_prepare_kernel<float><<<p.tokens, 128, 0, s>>>(p);
  else latent_prepare_kernel<bf16><<<p.tokens, 128, 0, s>>>(p);
  cuda_check(cudaGetLastError(), "latent_prepare_kernel");
}

void head_gate(const void* o, long long o_h, long long o_t, const void* gate, long long ld_gate, void* out, long long ld_out, int tokens, int H,
               int dv, int cols, int f32, cudaStream_t s) {
  if (tokens <= 0) return;
  if (f32)
    head_gate_kernel<float><<<tokens, 256, 0, s>>>(static_cast<const float*>(o), o_h, o_t, static_cast<const float*>(gate), ld_gate,
                                                   static_cast<float*>(out), ld_out, H, dv, cols);
  else
    head_gate_kernel<bf16><<<tokens, 256, 0, s>>>(static_cast<const bf16*>(o), o_h, o_t, static_cast<const bf16*>(gate), ld_gate,
                                                  static_cast<bf16*>(out), ld_out, H, dv, cols);
  cuda_check(cudaGetLastError(), "head_gate_kernel");
}

}  // namespace fllm
