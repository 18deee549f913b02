// Spread attention on the tensor cores, and the mixing of its heads (talking heads). A query head attends to the keys of its
// own key/value head with a sliding window and a distance bias, and weighs the values of every key/value head, which one cache row per
// token holds side by side:
//   s_j = scale q . k_j - r1 ln(1 + r2 (i - j)),   A = sum_j exp(s_j - m) v_j  (all heads' values),   l = sum_j exp(s_j - m)
// The fp32 partial sums (A, m, l) go to memory; talk_mix joins the key slices of a head and its sink and forms the heads' outputs
//   out_h = sigmoid(gate_h) sum_f talk[h, f] A_f(values of h's group) / (l_f + exp(sink_f - m_f))
// which equals mixing the heads' weights in front of the values.
//
// talk_prefill_kernel: one stream of 128 query rows (token * group + head) of one key head per CTA and up to 256 value columns. Warps 0 and 2
// bring tiles of 128 keys by TMA, warp 1 their values, all columns of a 16-token page in one box (issuing a box takes its thread as long as
// an MMA takes the tensor cores, whatever its size): a lane per page finds its place in the pool, one lane issues. Warp 3 issues the
// MMAs. Eight warps are the softmax: a row belongs to two threads with 64 columns each, which stay in registers between the maximum
// and the weights. Tensor memory: two score / weight buffers of 128 columns and 256 columns of output, so that the softmax of a tile runs
// under the products of the one before and the scores of the one after it. The weights travel as two bf16 terms, as in attention_maps.cu.
//
// talk_decode_kernel: mma.sync, 16 query rows (token * heads + head, so usually all heads of a token) and up to 256 value columns per CTA.
// The scores of all key heads fall into one accumulator: a row's queries are zero against every key head but its own. Each warp streams
// its own 16-token pages, the keys head by head and then the values in pieces, through a private cp.async ring; split over key slices.
//
// The bias enters as a factor: exp(s - bias_d) = exp(s - bias_d0) 2^-(bias_d - bias_d0), with d0 the smallest distance between the
// stream's tokens and the tile's, and the factors of all distances in a table that is made anew for every tile. The reference of a row is
// then at most the change of the bias inside a tile too high, which is why that change is limited (kTalkBiasRange). (Decode: as it is.)
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <algorithm>
#include <stdexcept>

#include "attention_util.cuh"
#include "fllm_ops.h"
#include "ptx.cuh"
#include "tma_host.h"

namespace fllm {
namespace {
constexpr float kLn2 = 0.6931471805599453f;
constexpr int kParts = 2, kSpan = kTile / kParts;        // threads of a row, columns of each
constexpr int kMmaWarp = 3, kFirstSoftmax = 128, kSoftmax = kRows * kParts, kThreads = kFirstSoftmax + kSoftmax;
constexpr int kCols = 256;                               // most value columns of a CTA
constexpr int kPiece = 128;                              // value columns of an item of the decode kernel's ring
constexpr int kTable = 2592;                             // fp32 entries of a tile's factors (16 heads of a group)
constexpr int kVStages = 3, kVPages = 4;                 // V comes in stages of four pages

struct Talk {
  const bf16 *q, *kc, *vc;
  const int* block_tables;
  int max_blocks;
  const int *q_starts, *positions;
  int H, G, group, block_size, window, wv;
  float scale_log2;
  const float *r1, *r2;
  float *part_o, *part_ml;
  int tab_stride, tab_entries, tab_bufs;                 // [buffer][head of the group][stride]
  int* status;
};

template <int DK>
struct TalkTile {
  static constexpr int kQ = tile_bytes<DK>(), kK = tile_bytes<DK>(), kV = kVPages * kPage * kCols * 2;
  static constexpr int kTail = 256 + 2 * kParts * kRows * 4 + kParts * kRows * 4 + 4 * 16 * 4 + kTable * 4;
  static constexpr int kTotal = kQ + 2 * kK + kVStages * kV + kTail + 1024;
  static_assert(kTotal <= 227 * 1024, "shared memory");
};

__device__ __forceinline__ void softmax_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(kSoftmax) : "memory"); }
// two fp32 operations at once
__device__ __forceinline__ uint64_t pair(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpair(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

__device__ __forceinline__ float lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float max3(float a, float b, float c) {
  float y;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(y) : "f"(a), "f"(b), "f"(c));
  return y;
}

// weights of kSpan columns of a row: sa holds the raw scores; columns [lo, hi) are visible (FULL: all); fac[-c] is the factor of column c.
// A weight is cut after its leading bf16 term, the second term is the rounded rest.
template <bool FULL>
__device__ __forceinline__ float weigh(uint32_t t_s, const uint32_t (&sa)[kSpan / 32][32], float scale_log2, float ref, const float* fac, int lo, int hi) {
  const uint64_t sc = pair(scale_log2, scale_log2), off = pair(-ref, -ref), minus = pair(-1.f, -1.f);
  uint64_t sum[2] = {0, 0};
#pragma unroll
  for (int b = 0; b < kSpan / 32; ++b) {
    uint32_t ph[16], pl[16];
#pragma unroll
    for (int i = 0; i < 32; i += 2) {
      const int c = 32 * b + i;
      const float2 t = unpair(fma2(pair(__uint_as_float(sa[b][i]), __uint_as_float(sa[b][i + 1])), sc, off));
      uint64_t v = mul2(pair(ex2(t.x), ex2(t.y)), pair(fac[-c], fac[-c - 1]));
      if (!FULL) {
        float2 w = unpair(v);
        if (c < lo || c >= hi) w.x = 0.f;
        if (c + 1 < lo || c + 1 >= hi) w.y = 0.f;
        v = pair(w.x, w.y);
      }
      sum[(i >> 1) & 1] = add2(sum[(i >> 1) & 1], v);
      const float2 w = unpair(v);
      const uint32_t x = __float_as_uint(w.x), y = __float_as_uint(w.y);
      ph[i / 2] = __byte_perm(x, y, 0x7632);
      const float2 rest = unpair(fma2(pair(__uint_as_float(x & 0xffff0000u), __uint_as_float(y & 0xffff0000u)), minus, v));
      pl[i / 2] = pack_bf16x2(rest.x, rest.y);
    }
    tmem_st_32x16(t_s + 32 * b, ph);
    tmem_st_32x16(t_s + 32 * b + 16, pl);
  }
  const float2 all = unpair(add2(sum[0], sum[1]));
  return all.x + all.y;
}
// the largest of kSpan scores, or of the visible ones
template <bool FULL>
__device__ __forceinline__ float largest(const uint32_t (&sa)[kSpan / 32][32], int lo, int hi) {
  auto at = [&](int c) { return FULL || (c >= lo && c < hi) ? __uint_as_float(sa[c >> 5][c & 31]) : -INFINITY; };
  float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
  for (int c = 0; c < kSpan; c += 2) mx[(c >> 1) & 3] = max3(mx[(c >> 1) & 3], at(c), at(c + 1));
  return fmaxf(max3(mx[0], mx[1], mx[2]), mx[3]);
}

// MN-major operand of 16 tokens: 1024 bytes between groups of eight tokens, 2048 between 64-column parts
__device__ __forceinline__ uint64_t desc_page(uint32_t saddr) {
  return (uint64_t)((saddr & 0x3FFFFu) >> 4) | (uint64_t)(kPage * 128 >> 4) << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}

template <int DK>
__global__ void __launch_bounds__(kThreads, 1) talk_prefill_kernel(const __grid_constant__ CUtensorMap tma_k, const __grid_constant__ CUtensorMap tma_v,
                                                                   const Talk p, int min_rows, int col_ctas) {
  using L = TalkTile<DK>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sq = smem;
  uint8_t* sk = smem + L::kQ;                                        // [2]
  uint8_t* sv = sk + 2 * L::kK;                                      // [kVStages][page][64-column part][token], 128-byte swizzled rows
  uint64_t* bars = reinterpret_cast<uint64_t*>(sv + kVStages * L::kV);
  uint64_t *k_full = bars, *k_empty = bars + 2, *s_full = bars + 4, *p_ready = bars + 6, *o_done = bars + 7, *q_full = bars + 31;
  uint64_t *v_full = bars + 8, *v_empty = bars + 8 + kVStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8 + 2 * kVStages);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* swap_m = reinterpret_cast<float*>(bars + 32);               // [buffer][part][row]
  float* swap_l = swap_m + 2 * kParts * kRows;                       // [part][row]
  float* rates = swap_l + kParts * kRows;                                 // [head of the group] r1, then r2
  float* near_bias = rates + 2 * 16;                                 // [buffer][head of the group]: bias of a tile's smallest distance
  float* table = near_bias + 2 * 16;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row0 = (gridDim.x - 1 - blockIdx.x) * kRows;             // the tiles with the longest key range start first
  const int kvh = blockIdx.y / col_ctas, col0 = blockIdx.y % col_ctas * kCols, seq = blockIdx.z;
  const int cols = min(kCols, p.wv - col0), v_page = kPage * 2 * min(kCols, p.wv);      // bytes of a page as it is fetched (zeros beyond the row)
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0;
  const int all_rows = qn * p.group;
  if (all_rows < min_rows || row0 >= all_rows) return;
  const int kv_len = p.positions[q0 + qn - 1] + 1, first_pos = kv_len - qn;
  const int n_rows = min(kRows, all_rows - row0), i0 = first_pos + row0 / p.group;
  const int first = p.window > 0 ? max(0, i0 + 1 - p.window) : 0, begin = first / kPage * kPage;
  const int n_tiles = (first_pos + (row0 + n_rows - 1) / p.group + 1 - begin + kTile - 1) / kTile;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) mbar_init(&k_full[i], 2), mbar_init(&k_empty[i], 1), mbar_init(&s_full[i], 1);
    for (int i = 0; i < kVStages; ++i) mbar_init(&v_full[i], 1), mbar_init(&v_empty[i], 1);
    mbar_init(p_ready, kSoftmax / 32), mbar_init(o_done, 1), mbar_init(q_full, kSoftmax);
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (threadIdx.x == 0) tma_prefetch_desc(&tma_k);
  if (threadIdx.x == 32) tma_prefetch_desc(&tma_v);
  if (warp == kMmaWarp) tmem_alloc(tmem_slot, 512), tmem_relinquish();
  auto bias = [](float a, float b, int d) { return a * lg2(fmaf(b, (float)d, 1.f)); };
  auto nearest = [&](int it) { return max(i0 - (begin + it * kTile) - (kTile - 1), 0); };
  if (threadIdx.x < p.group) {
    const int head = kvh * p.group + threadIdx.x;
    const float a = p.r1 ? p.r1[head] : 0.f, b = p.r1 ? p.r2[head] : 0.f;
    rates[threadIdx.x] = a, rates[16 + threadIdx.x] = b, near_bias[threadIdx.x] = bias(a, b, nearest(0));
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp < kMmaWarp) {
    constexpr int PAGES = kTile / kPage;
    const int* blocks = p.block_tables + (size_t)seq * p.max_blocks;
    const int last = (kv_len - 1) / kPage * kPage;                     // pages past the sequence repeat its last one (finite values)
    // of the lane's page in tile `it`: its first row, in a pool of `heads` rows per token
    auto first_row = [&](int it, int heads, int head) {
      const int tok = min(begin + it * kTile + lane % PAGES * kPage, last);
      return (blocks[tok / p.block_size] * heads + head) * p.block_size + tok % p.block_size;
    };
    if (warp != 1) {                                                   // half of the pages' keys
      const int pg0 = warp == 0 ? 0 : PAGES / 2;
      int row = first_row(0, p.G, kvh);
      for (int it = 0; it < n_tiles; ++it) {
        const int now = row, b = it & 1, use = it >> 1;
        if (it + 1 < n_tiles) row = first_row(it + 1, p.G, kvh);
        if (!__all_sync(0xffffffffu, use == 0 || mbar_wait(&k_empty[b], (use - 1) & 1, abort_flag))) break;
        if (lane == 0) mbar_expect_tx(&k_full[b], tile_bytes<DK>() / 2);
#pragma unroll
        for (int pg = 0; pg < PAGES / 2; ++pg) {
          const int y = __shfl_sync(0xffffffffu, now, pg0 + pg);
          if (lane == 0) {
#pragma unroll
            for (int h = 0; h < DK / 64; ++h) tma_load_2d(sk + b * L::kK + h * kHalf + (pg0 + pg) * (kPage * 128), &tma_k, &k_full[b], 64 * h, y);
          }
        }
      }
    } else {
      int row = first_row(0, 1, 0), vs = 0, v_use = 0;
      bool ok = true;
      for (int it = 0; ok && it < n_tiles; ++it) {
        const int now = row;
        if (it + 1 < n_tiles) row = first_row(it + 1, 1, 0);
#pragma unroll 1
        for (int c = 0; c < PAGES; c += kVPages) {
          if (!(ok = __all_sync(0xffffffffu, v_use == 0 || mbar_wait(&v_empty[vs], (v_use - 1) & 1, abort_flag)))) break;
          if (lane == 0) mbar_expect_tx(&v_full[vs], kVPages * v_page);
#pragma unroll
          for (int pg = 0; pg < kVPages; ++pg) {
            const int y = __shfl_sync(0xffffffffu, now, c + pg);
            if (lane == 0) tma_load_3d(sv + vs * L::kV + pg * v_page, &tma_v, &v_full[vs], 0, y, col0 / 64);
          }
          if (++vs == kVStages) vs = 0, ++v_use;
        }
      }
    }
  } else if (warp == kMmaWarp) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc(128, 128, 1, 1);
      const uint32_t idesc_pv = make_idesc(128, cols, 1, 1) | (1u << 16);      // B is MN-major
      const uint32_t q_addr = smem_u32(sq), k_addr = smem_u32(sk), v_addr = smem_u32(sv);
      bool ok = true;
      auto scores = [&](int it) {
        const int b = it & 1;
        if (!(ok = mbar_wait(&k_full[b], (it >> 1) & 1, abort_flag))) return;
        tc_fence_after_sync();
#pragma unroll
        for (int k = 0; k < DK / 16; ++k) {
          const uint32_t off = (k >> 2) * kHalf + (k & 3) * 32;
          tc_mma_bf16(tmem_base + 128 * b, make_smem_desc_sw128(q_addr + off), make_smem_desc_sw128(k_addr + b * L::kK + off), idesc_s, k > 0);
        }
        tc_commit(&s_full[b]);
        tc_commit(&k_empty[b]);
      };
      ok = mbar_wait(q_full, 0, abort_flag);
      if (ok) scores(0);
      if (ok && n_tiles > 1) scores(1);
      int vs = 0, v_use = 0;
      for (int it = 0; ok && it < n_tiles; ++it) {
        const uint32_t t_p = tmem_base + 128 * (it & 1);
        if (!(ok = mbar_wait(p_ready, it & 1, abort_flag))) break;
        for (int c = 0; c < kTile / kPage; c += kVPages) {
          if (!(ok = mbar_wait(&v_full[vs], v_use & 1, abort_flag))) break;
          tc_fence_after_sync();
#pragma unroll
          for (int pg = 0; pg < kVPages; ++pg) {
            const int k = c + pg;
            const uint32_t a = t_p + 32 * (k >> 1) + 8 * (k & 1);
            const uint64_t v = desc_page(v_addr + vs * L::kV + pg * v_page);
            tc_mma_bf16_ts(tmem_base + 256, a, v, idesc_pv, it > 0 || k > 0);
            tc_mma_bf16_ts(tmem_base + 256, a + 16, v, idesc_pv, 1);
          }
          tc_commit(&v_empty[vs]);
          if (++vs == kVStages) vs = 0, ++v_use;
        }
        if (!ok) break;
        tc_commit(o_done);
        if (it + 2 < n_tiles) scores(it + 2);
      }
    }
  } else if (warp >= kFirstSoftmax / 32) {                             // (warp 2 has no work)
    // thread of a row's columns kSpan part .. + kSpan - 1; the row is in the lane quarter this warp may touch
    const int part = (warp - kFirstSoftmax / 32) >> 2, r = (warp & 3) * 32 + lane, id = threadIdx.x - kFirstSoftmax;
    // the query rows go to shared memory in the layout TMA's 128-byte swizzle would have produced, all loads of a thread in flight at once
    {
      constexpr int CHUNKS = DK / 8, STEP = kSoftmax / CHUNKS, N = kRows / STEP;
      const int c = id % CHUNKS;
      uint4 v[N];
#pragma unroll
      for (int k = 0; k < N; ++k) {
        const int row = row0 + id / CHUNKS + k * STEP, tok = row / p.group;
        v[k] = make_uint4(0, 0, 0, 0);
        if (row < all_rows) v[k] = *reinterpret_cast<const uint4*>(p.q + ((long long)(q0 + tok) * p.H + kvh * p.group + row - tok * p.group) * DK + c * 8);
      }
#pragma unroll
      for (int k = 0; k < N; ++k) {
        const int rr = id / CHUNKS + k * STEP;
        *reinterpret_cast<uint4*>(sq + (c >> 3) * kHalf + rr * 128 + (((c & 7) ^ (rr & 7)) << 4)) = v[k];
      }
      fence_proxy_async_smem();
      mbar_arrive(q_full);
    }
    const uint32_t lane_off = (uint32_t)((warp & 3) * 32) << 16;
    const bool valid = r < n_rows;
    const int lim = valid ? first_pos + (row0 + r) / p.group + 1 : 0, beg = p.window > 0 ? max(0, lim - p.window) : 0;
    const int last_lim = first_pos + (row0 + n_rows - 1) / p.group + 1, beg_last = p.window > 0 ? max(0, last_lim - p.window) : 0;
    const int off = (row0 + r) / p.group - row0 / p.group, hh = (row0 + r) % p.group;      // token behind the CTA's first, head of the group
    const int e_head = id / p.tab_stride, e_at = id % p.tab_stride, jump_head = kSoftmax / p.tab_stride, jump_at = kSoftmax % p.tab_stride;
    float* my_max = swap_m + r;
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int it = 0; it < n_tiles; ++it) {
      const int tok0 = begin + it * kTile, base = i0 - tok0 - (kTile - 1), d0 = max(base, 0);
      // factors of the distances base + e, e = off + 127 - column
      float* buf = table + (p.tab_bufs == 2 && (it & 1) ? p.tab_entries : 0);
      if (p.tab_bufs == 1 && it > 0) softmax_barrier();
      for (int head = e_head, at = e_at, i = id; i < p.tab_entries; i += kSoftmax) {
        buf[i] = ex2(near_bias[(it & 1) * 16 + head] - bias(rates[head], rates[16 + head], max(base + at, d0)));
        head += jump_head, at += jump_at;
        if (at >= p.tab_stride) at -= p.tab_stride, ++head;
      }
      const float b0 = near_bias[(it & 1) * 16 + hh];
      if (id < p.group) near_bias[(~it & 1) * 16 + id] = bias(rates[id], rates[16 + id], nearest(it + 1));
      const uint32_t t_s = tmem_base + 128 * (it & 1) + kSpan * part + lane_off;
      // every thread waits for every tile's output products, in order: before it touches the output, or at its end
      bool waited = it == 0;
      auto wait_output = [&]() {
        if (waited) return;
        if (!mbar_wait(o_done, (it - 1) & 1, abort_flag)) ok = false;
        tc_fence_after_sync();
        waited = true;
      };
      if (!mbar_wait(&s_full[it & 1], (it >> 1) & 1, abort_flag)) ok = false;
      tc_fence_after_sync();
      uint32_t sa[kSpan / 32][32];
#pragma unroll
      for (int b = 0; b < kSpan / 32; ++b) tmem_ld_32x32(t_s + 32 * b, sa[b]);
      tmem_ld_wait();
      const int lo = beg - tok0 - kSpan * part, hi = lim - tok0 - kSpan * part;
      const bool full = n_rows == kRows && tok0 + kTile <= i0 + 1 && tok0 >= beg_last;
      float* row_max = my_max + (it & 1) * kParts * kRows;
      row_max[part * kRows] = full ? largest<true>(sa, 0, 0) : largest<false>(sa, lo, hi);
      softmax_barrier();
      float raw = row_max[0];
#pragma unroll
      for (int k = 1; k < kParts; ++k) raw = fmaxf(raw, row_max[k * kRows]);
      const float top = raw == -INFINITY ? -INFINITY : fmaf(raw, p.scale_log2, -b0);
      // a row keeps its old reference unless the new maximum is far above it; the decision is per warp because the tensor
      // memory accesses of the rescale are warp-wide, and all warps of the rows take the same one
      if (__any_sync(0xffffffffu, top > m_used + kLazyRescale || (m_used == -INFINITY && top > -INFINITY))) {
        const float m_new = fmaxf(m_used, top), corr = m_new == -INFINITY ? 1.f : ex2(m_used - m_new);
        m_used = m_new;
        l *= corr;
        if (it > 0) {
          wait_output();
#pragma unroll 1
          for (int c = part * 32; c < cols; c += 32 * kParts) {
            uint32_t o[32];
            const uint32_t t_o = tmem_base + 256 + c + lane_off;
            tmem_ld_32x32(t_o, o);
            tmem_ld_wait();
            uint32_t a[16], b[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              a[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
              b[i] = __float_as_uint(__uint_as_float(o[16 + i]) * corr);
            }
            tmem_st_32x16(t_o, a);
            tmem_st_32x16(t_o + 16, b);
          }
        }
      }
      const float ref = (m_used == -INFINITY ? 0.f : m_used) + b0;
      const float* fac = buf + hh * p.tab_stride + off + (kTile - 1) - kSpan * part;
      l += full ? weigh<true>(t_s, sa, p.scale_log2, ref, fac, 0, 0) : weigh<false>(t_s, sa, p.scale_log2, ref, fac, lo, hi);
      tmem_st_wait();
      wait_output();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    ok = ok && mbar_wait(o_done, (n_tiles - 1) & 1, abort_flag);
    tc_fence_after_sync();
    swap_l[part * kRows + r] = l;
    softmax_barrier();
    l = 0.f;
#pragma unroll
    for (int k = 0; k < kParts; ++k) l += swap_l[k * kRows + r];
    // blocks of 32 rows x 32 columns go out through shared memory (the keys' place), so that eight lanes write 128 bytes of a row
    constexpr int LD = 36;
    static_assert(2 * L::kK + kVStages * L::kV >= kSoftmax / 32 * 32 * LD * 4, "room for the output blocks");
    float* turn = reinterpret_cast<float*>(sk) + (warp - kFirstSoftmax / 32) * (32 * LD);
    long long to[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const int row = row0 + (warp & 3) * 32 + 4 * k + lane / 8, tok = row / p.group;
      to[k] = ok && row < all_rows ? ((long long)(q0 + tok) * p.H + kvh * p.group + row - tok * p.group) * p.wv + col0 + 4 * (lane % 8) : -1;
    }
#pragma unroll 1
    for (int c = part * 32; c < cols; c += 32 * kParts) {
      uint32_t o[32];
      tmem_ld_32x32(tmem_base + 256 + c + lane_off, o);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; i += 4) *reinterpret_cast<uint4*>(turn + lane * LD + i) = make_uint4(o[i], o[i + 1], o[i + 2], o[i + 3]);
      __syncwarp();
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float4 v = *reinterpret_cast<const float4*>(turn + (4 * k + lane / 8) * LD + 4 * (lane % 8));
        if (to[k] >= 0) *reinterpret_cast<float4*>(p.part_o + to[k] + c) = v;
      }
      __syncwarp();
    }
    const int row = row0 + r;
    const long long at = (long long)(q0 + row / p.group) * p.H + kvh * p.group + row % p.group;
    if (ok && valid && part == 0 && col0 == 0) p.part_ml[2 * at] = m_used * kLn2, p.part_ml[2 * at + 1] = l;
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == kMmaWarp) { tc_fence_after_sync(); tmem_dealloc(tmem_base, 512); }
  if (threadIdx.x == 0 && *abort_flag && p.status) atomicCAS(p.status, FLLM_OK, FLLM_ERR_MBAR_TIMEOUT);
}

// ------------------------------------------------------------------------------------------ decode
constexpr int kDecodeRows = 64;           // sequences with at most this many query rows per key head run here
constexpr int kSlots = 6, kSlot = 4096;   // a warp's ring: one key head, or 128 value columns, of a page each
template <int DK, int NC>
struct TalkDecode {
  static constexpr int kQ = 16 * DK * 2, kRing = 4 * kSlots * kSlot, kMerge = 4 * 16 * NC * 4 + 4 * 16 * 2 * 4;
  static constexpr int kTotal = kQ + (kRing > kMerge ? kRing : kMerge) + 128;
};

template <int DK, int NC>
__global__ void __launch_bounds__(128, 2) talk_decode_kernel(const Talk p, int col_ctas, int splits) {
  using L = TalkDecode<DK, NC>;
  constexpr int DV = NC < kPiece ? NC : kPiece, PIECES = NC / DV;
  extern __shared__ __align__(128) uint8_t smem[];
  bf16* qtile = reinterpret_cast<bf16*>(smem);
  uint8_t* ring = smem + L::kQ;
  const int row0 = blockIdx.x / col_ctas * 16, col0 = blockIdx.x % col_ctas * NC, seq = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, H = p.H;
  pdl_launch_dependents();
  pdl_wait();
  const int q0 = p.q_starts[seq], qn = p.q_starts[seq + 1] - q0;
  const int all_rows = qn * H;
  if (qn <= 0 || qn * p.group > kDecodeRows || row0 >= all_rows) return;
  const int n_rows = min(16, all_rows - row0), last_row = row0 + n_rows - 1;
  const int kv_len = p.positions[q0 + qn - 1] + 1, first_pos = kv_len - qn;
  const int hi_tok = first_pos + last_row / H + 1, first = p.window > 0 ? max(0, first_pos + row0 / H + 1 - p.window) : 0;
  const int page0 = first / kPage, pages = (hi_tok + kPage - 1) / kPage - page0, per = (pages + splits - 1) / splits;
  const int pg0 = page0 + split * per, pg1 = page0 + min((split + 1) * per, pages);
  // key heads of these rows
  const bool one = row0 / H == last_row / H;
  const int g_lo = one ? row0 % H / p.group : 0, heads = (one ? last_row % H / p.group : p.G - 1) - g_lo + 1;
  const int items = heads + PIECES;                       // of a page

  for (int i = threadIdx.x; i < 16 * (DK / 8); i += 128) {
    const int r = i / (DK / 8), c = i - r * (DK / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < n_rows) v = *reinterpret_cast<const uint4*>(p.q + ((long long)(q0 + (row0 + r) / H) * H + (row0 + r) % H) * DK + c * 8);
    *reinterpret_cast<uint4*>(tile_ptr<DK>(qtile, r, c)) = v;
  }
  __syncthreads();
  uint32_t qf[DK / 16][4];
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk) ldsm_x4(qf[kk], tile_ptr<DK>(qtile, lane & 15, 2 * kk + (lane >> 4)));

  const int t4 = lane & 3;
  int lim[2], beg[2], own[2];
  float r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = (lane >> 2) + 8 * i, head = (row0 + r) % H;
    lim[i] = r < n_rows ? first_pos + (row0 + r) / H + 1 : 0;
    beg[i] = p.window > 0 ? max(0, lim[i] - p.window) : 0;
    own[i] = head / p.group - g_lo;
    if (p.r1) r1[i] = p.r1[head], r2[i] = p.r2[head];
  }
  float o[NC / 8][4];
#pragma unroll
  for (int i = 0; i < NC / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};

  uint8_t* mine = ring + (size_t)warp * kSlots * kSlot;
  const int* table = p.block_tables + (size_t)seq * p.max_blocks;
  const int my_pages = pg1 > pg0 + warp ? (pg1 - pg0 - warp + 3) / 4 : 0;
  // the next item to fetch: item in_item of the page at block in_block, in_at
  int in_left = my_pages, in_page = pg0 + warp, in_item = 0, in_slot = 0, in_block = 0, in_at = 0;
  auto issue = [&]() {
    if (in_left > 0) {
      if (in_item == 0) in_block = table[in_page * kPage / p.block_size], in_at = in_page * kPage % p.block_size;
      bf16* dst = reinterpret_cast<bf16*>(mine + in_slot * kSlot);
      if (in_item < heads) {
        const bf16* src = p.kc + ((long long)(in_block * p.G + g_lo + in_item) * p.block_size + in_at) * DK;
#pragma unroll
        for (int i = lane; i < kPage * (DK / 8); i += 32) cp_async16(tile_ptr<DK>(dst, i / (DK / 8), i % (DK / 8)), src + i * 8);
      } else {
        const bf16* src = p.vc + ((long long)in_block * p.block_size + in_at) * p.wv + col0 + (in_item - heads) * DV;
#pragma unroll
        for (int i = lane; i < kPage * (DV / 8); i += 32)
          cp_async16(tile_ptr<DV>(dst, i / (DV / 8), i % (DV / 8)), src + (size_t)(i / (DV / 8)) * p.wv + i % (DV / 8) * 8);
      }
      if (++in_item == items) in_item = 0, in_page += 4, --in_left;
    }
    if (++in_slot == kSlots) in_slot = 0;
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < kSlots - 1; ++i) issue();
  int slot = 0;
  // the slot of the next item, its bytes complete; the slot of the item before it is fetched into again
  auto next = [&]() {
    __syncwarp();
    issue();
    cp_async_wait<kSlots - 1>();
    __syncwarp();
    bf16* at = reinterpret_cast<bf16*>(mine + slot * kSlot);
    if (++slot == kSlots) slot = 0;
    return at;
  };
  const int j4 = lane >> 3;
  for (int it = 0; it < my_pages; ++it) {
    const int tok_base = (pg0 + warp + 4 * it) * kPage;
    float s[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    for (int g = 0; g < heads; ++g) {
      bf16* ks = next();
      const uint32_t lo = own[0] == g ? 0xffffffffu : 0u, hi = own[1] == g ? 0xffffffffu : 0u;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        const uint32_t a[4] = {qf[kk][0] & lo, qf[kk][1] & hi, qf[kk][2] & lo, qf[kk][3] & hi};
        uint32_t b[4];
        ldsm_x4(b, tile_ptr<DK>(ks, (j4 >> 1) * 8 + (lane & 7), 2 * kk + (j4 & 1)));
        mma_bf16(s[0], a, b[0], b[1]);
        mma_bf16(s[1], a, b[2], b[3]);
      }
    }
    // ---- weights of two rows x four tokens
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = e >> 1, tok = tok_base + nb * 8 + 2 * t4 + (e & 1);
        const float v = s[nb][e] * p.scale_log2 - r1[i] * __log2f(fmaf(r2[i], (float)(lim[i] - 1 - tok), 1.f));
        s[nb][e] = tok >= beg[i] && tok < lim[i] ? v : -INFINITY;
        mx[i] = fmaxf(mx[i], s[nb][e]);
      }
    }
    float ref[2], c[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
      const float mn = fmaxf(m[i], mx[i]);
      ref[i] = mn == -INFINITY ? 0.f : mn;
      c[i] = ex2(m[i] - ref[i]);
      l[i] *= c[i];
      m[i] = mn;
    }
    if (__any_sync(0xffffffffu, c[0] != 1.f || c[1] != 1.f)) {
#pragma unroll
      for (int db = 0; db < NC / 8; ++db) o[db][0] *= c[0], o[db][1] *= c[0], o[db][2] *= c[1], o[db][3] *= c[1];
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
    for (int piece = 0; piece < PIECES; ++piece) {
      bf16* vs = next();
#pragma unroll
      for (int db = 0; db < DV / 8; db += 2) {
        uint32_t b[4];
        ldsm_x4_t(b, tile_ptr<DV>(vs, (j4 & 1) * 8 + (lane & 7), db + (j4 >> 1)));
        float(&o0)[4] = o[piece * (DV / 8) + db];
        float(&o1)[4] = o[piece * (DV / 8) + db + 1];
        mma_bf16(o0, ph, b[0], b[1]);
        mma_bf16(o1, ph, b[2], b[3]);
        mma_bf16(o0, pl, b[0], b[1]);
        mma_bf16(o1, pl, b[2], b[3]);
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
  }
  __syncthreads();                                       // the rings are free: merge the four warps
  float* mo = reinterpret_cast<float*>(smem + L::kQ);    // [4][16][NC]
  float* mml = mo + 4 * 16 * NC;                         // [4][16][2]
  const int g8 = lane >> 2;
#pragma unroll
  for (int db = 0; db < NC / 8; ++db) {
    *reinterpret_cast<float2*>(mo + ((size_t)warp * 16 + g8) * NC + db * 8 + 2 * t4) = make_float2(o[db][0], o[db][1]);
    *reinterpret_cast<float2*>(mo + ((size_t)warp * 16 + g8 + 8) * NC + db * 8 + 2 * t4) = make_float2(o[db][2], o[db][3]);
  }
  if (t4 == 0) {
#pragma unroll
    for (int i = 0; i < 2; ++i) mml[(warp * 16 + g8 + 8 * i) * 2] = m[i], mml[(warp * 16 + g8 + 8 * i) * 2 + 1] = l[i];
  }
  __syncthreads();
  for (int r = warp; r < n_rows; r += 4) {
    float ms = -INFINITY, ls = 0.f, c[4];
#pragma unroll
    for (int w = 0; w < 4; ++w) ms = fmaxf(ms, mml[(w * 16 + r) * 2]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = mml[(w * 16 + r) * 2];
      c[w] = mw == -INFINITY ? 0.f : ex2(mw - ms);
      ls = fmaf(mml[(w * 16 + r) * 2 + 1], c[w], ls);
    }
    const size_t at = ((size_t)q0 * H + row0 + r) * splits + split;
#pragma unroll
    for (int e = 0; e < NC / 32; ++e) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) v = fmaf(mo[((size_t)w * 16 + r) * NC + lane + 32 * e], c[w], v);
      if (col0 + lane + 32 * e < p.wv) p.part_o[at * p.wv + col0 + lane + 32 * e] = v;
    }
    if (lane == 0 && col0 == 0) p.part_ml[at * 2] = ms * kLn2, p.part_ml[at * 2 + 1] = ls;
  }
}

// ------------------------------------------------------------------------------------------ mixing
// One key slice per head (prompts, and batches that fill the GPU): a thread has four value columns of a token and mixes four heads at a
// time, blockDim.y tokens per CTA.
template <typename T>
__global__ void __launch_bounds__(256) talk_mix_rows_kernel(const TalkMixParams p) {
  extern __shared__ float sm[];
  const int H = p.H, group = H / p.G, t = blockIdx.x * blockDim.y + threadIdx.y, id = threadIdx.y * blockDim.x + threadIdx.x, n = blockDim.x * blockDim.y;
  float* mat = sm;                             // [f][h]
  float* coef = sm + H * H + threadIdx.y * H;
  pdl_launch_dependents();
  for (int i = id; i < H * H; i += n) mat[i % H * H + i / H] = p.talk[i];
  pdl_wait();
  if (t < p.tokens)
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
      const float2 v = __ldcg(reinterpret_cast<const float2*>(p.part_ml) + (size_t)t * H + h);
      coef[h] = 1.f / (v.y + (p.sink ? expf(p.sink[h] - v.x) : 0.f));
    }
  __syncthreads();
  if (t >= p.tokens) return;
  T* out = static_cast<T*>(p.out) + (long long)t * p.ldo;
  for (int c = 4 * threadIdx.x; c < p.G * p.v_dim; c += 4 * blockDim.x) {
    const int g = c / p.v_dim, i = c - g * p.v_dim;
    const float* src = p.part_o + (size_t)t * H * p.wv + c;
    for (int e0 = 0; e0 < group; e0 += 4) {
      const int h0 = g * group + e0, k = min(4, group - e0);
      float4 acc[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[e] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (int f = 0; f < H; ++f) {
        float4 a = __ldcg(reinterpret_cast<const float4*>(src + (size_t)f * p.wv));
        const float z = coef[f];
        a.x *= z, a.y *= z, a.z *= z, a.w *= z;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float w = mat[f * H + h0 + min(e, k - 1)];
          acc[e].x = fmaf(w, a.x, acc[e].x), acc[e].y = fmaf(w, a.y, acc[e].y), acc[e].z = fmaf(w, a.z, acc[e].z), acc[e].w = fmaf(w, a.w, acc[e].w);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (e >= k) continue;
        const float z = p.gate ? 1.f / (1.f + expf(-p.gate[(long long)t * p.ld_gate + h0 + e])) : 1.f;
        const float v[4] = {acc[e].x * z, acc[e].y * z, acc[e].z * z, acc[e].w * z};
        T* to = out + (long long)(h0 + e) * p.v_dim + i;
        if (p.vec) {
          typename Four<T>::type raw;
          T* x = reinterpret_cast<T*>(&raw);
#pragma unroll
          for (int j = 0; j < 4; ++j) x[j] = from_f32<T>(v[j]);
          *reinterpret_cast<typename Four<T>::type*>(to) = raw;
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j) to[j] = from_f32<T>(v[j]);
        }
      }
    }
  }
  for (int c = H * p.v_dim + threadIdx.x; c < p.cols; c += blockDim.x) out[c] = from_f32<T>(0.f);
}

// Several key slices, or few tokens: a CTA per token, blockDim.x threads with four columns each times blockDim.y shares of the heads, whose
// parts of four mixed heads are added up through shared memory.
template <typename T>
__global__ void __launch_bounds__(512) talk_mix_slices_kernel(const TalkMixParams p) {
  extern __shared__ __align__(16) float sm[];
  const int H = p.H, S = p.splits, group = H / p.G, t = blockIdx.x, X = blockDim.x, Y = blockDim.y, x = threadIdx.x, y = threadIdx.y;
  const int id = y * X + x, n = X * Y, warp = id >> 5, lane = id & 31;
  float4* part = reinterpret_cast<float4*>(sm);          // [4][Y][X]
  float* mat = sm + 16 * n;                              // [f][h]
  float* coef = mat + H * H;                             // [f][slice]
  pdl_launch_dependents();
  for (int i = id; i < H * H; i += n) mat[i % H * H + i / H] = p.talk[i];
  pdl_wait();
  for (int h = warp; h < H; h += n / 32) {               // a lane per key slice
    const float2 v = lane < S ? __ldcg(reinterpret_cast<const float2*>(p.part_ml) + ((size_t)t * H + h) * S + lane) : make_float2(-INFINITY, 0.f);
    const float m = warp_max(v.x), c = v.x == -INFINITY ? 0.f : expf(v.x - m), l = warp_sum(v.y * c) + (p.sink ? expf(p.sink[h] - m) : 0.f);
    if (lane < S) coef[h * S + lane] = c / l;
  }
  __syncthreads();
  T* out = static_cast<T*>(p.out) + (long long)t * p.ldo;
  const int cols = p.G * p.v_dim;
  for (int c0 = 0; c0 < cols; c0 += 4 * X) {
    const int c = c0 + 4 * x, g = min(c, cols - 4) / p.v_dim, i = c - g * p.v_dim;
    const float* src = p.part_o + (size_t)t * H * S * p.wv + c;
    for (int e0 = 0; e0 < group; e0 += 4) {
      const int h0 = g * group + e0, k = min(4, group - e0);
      float4 acc[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[e] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < cols) {
        for (int f = y; f < H; f += Y) {
          float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
          for (int s = 0; s < S; ++s) {
            const float4 v = __ldcg(reinterpret_cast<const float4*>(src + ((size_t)f * S + s) * p.wv));
            const float z = coef[f * S + s];
            a.x = fmaf(z, v.x, a.x), a.y = fmaf(z, v.y, a.y), a.z = fmaf(z, v.z, a.z), a.w = fmaf(z, v.w, a.w);
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float w = mat[f * H + h0 + min(e, k - 1)];
            acc[e].x = fmaf(w, a.x, acc[e].x), acc[e].y = fmaf(w, a.y, acc[e].y), acc[e].z = fmaf(w, a.z, acc[e].z), acc[e].w = fmaf(w, a.w, acc[e].w);
          }
        }
      }
      __syncthreads();
#pragma unroll
      for (int e = 0; e < 4; ++e) part[e * n + id] = acc[e];
      __syncthreads();
      for (int e = y; e < k && c < cols; e += Y) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int j = 0; j < Y; ++j) {
          const float4 q = part[e * n + j * X + x];
          v.x += q.x, v.y += q.y, v.z += q.z, v.w += q.w;
        }
        const float z = p.gate ? 1.f / (1.f + expf(-p.gate[(long long)t * p.ld_gate + h0 + e])) : 1.f;
        T* to = out + (long long)(h0 + e) * p.v_dim + i;
        to[0] = from_f32<T>(v.x * z), to[1] = from_f32<T>(v.y * z), to[2] = from_f32<T>(v.z * z), to[3] = from_f32<T>(v.w * z);
      }
    }
  }
  for (int c = H * p.v_dim + id; c < p.cols; c += n) out[c] = from_f32<T>(0.f);
}

// Any value width: one CTA per token and NC of its value columns (g, i), 256 / NC threads per column: the normalised column of every head's output is
// put together from its key slices, then each thread mixes some of the heads of group g.
constexpr int kMixHeads = 8;
template <typename T, int NC>
__global__ void __launch_bounds__(256) talk_mix_kernel(const TalkMixParams p) {
  constexpr int NF = 256 / NC;
  extern __shared__ float sm[];
  const int t = blockIdx.x, H = p.H, group = H / p.G, S = p.splits, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* coef = sm;                            // [H][S]
  float* a = coef + H * S;                     // [H][NC]
  pdl_launch_dependents();
  pdl_wait();
  if (S == 1) {
    for (int h = threadIdx.x; h < H; h += 256) {
      const float2 v = __ldcg(reinterpret_cast<const float2*>(p.part_ml) + (size_t)t * H + h);
      coef[h] = 1.f / (v.y + (p.sink ? expf(p.sink[h] - v.x) : 0.f));
    }
  } else {
    for (int h = warp; h < H; h += 8) {        // a lane per key slice
      const float2 v = lane < S ? __ldcg(reinterpret_cast<const float2*>(p.part_ml) + ((size_t)t * H + h) * S + lane) : make_float2(-INFINITY, 0.f);
      const float m = warp_max(v.x), c = v.x == -INFINITY ? 0.f : expf(v.x - m), l = warp_sum(v.y * c) + (p.sink ? expf(p.sink[h] - m) : 0.f);
      if (lane < S) coef[h * S + lane] = c / l;
    }
  }
  __syncthreads();
  const int slice = threadIdx.x / NC, c = blockIdx.y * NC + threadIdx.x % NC, cols = p.G * p.v_dim;
  if (c < cols) {
    const float* src = p.part_o + (size_t)t * H * S * p.wv + c;
    if (S == 1) {
#pragma unroll 8
      for (int f = slice; f < H; f += NF) a[f * NC + threadIdx.x % NC] = __ldcg(src + (size_t)f * p.wv) * coef[f];
    } else {
      for (int f = slice; f < H; f += NF) {
        float v = 0.f;
#pragma unroll 8
        for (int s = 0; s < S; ++s) {
          const float w = coef[f * S + s];     // (an empty slice may hold anything)
          const float o = __ldcg(src + ((size_t)f * S + s) * p.wv);
          v = w != 0.f ? fmaf(o, w, v) : v;
        }
        a[f * NC + threadIdx.x % NC] = v;
      }
    }
  }
  __syncthreads();
  T* out = static_cast<T*>(p.out) + (long long)t * p.ldo;
  if (c < cols) {
    const int g = c / p.v_dim, i = c - g * p.v_dim;
    for (int e0 = slice; e0 < group; e0 += NF * kMixHeads) {
      float acc[kMixHeads];
#pragma unroll
      for (int e = 0; e < kMixHeads; ++e) acc[e] = 0.f;
      const float* row = p.talk + (size_t)(g * group + e0) * H;
#pragma unroll 4
      for (int f = 0; f < H; ++f) {
        const float v = a[f * NC + threadIdx.x % NC];
#pragma unroll
        for (int e = 0; e < kMixHeads; ++e)
          if (e0 + e * NF < group) acc[e] = fmaf(__ldg(row + (size_t)e * NF * H + f), v, acc[e]);
      }
#pragma unroll
      for (int e = 0; e < kMixHeads; ++e) {
        const int h = g * group + e0 + e * NF;
        if (e0 + e * NF >= group) continue;
        const float z = p.gate ? 1.f / (1.f + expf(-p.gate[(long long)t * p.ld_gate + h])) : 1.f;
        out[(long long)h * p.v_dim + i] = from_f32<T>(acc[e] * z);
      }
    }
  }
  if (blockIdx.y == 0)
    for (int k = H * p.v_dim + threadIdx.x; k < p.cols; k += 256) out[k] = from_f32<T>(0.f);
}

template <typename T>
void launch_mix_slices(const TalkMixParams& p, cudaStream_t s) {
  const int x = std::min(128, (p.G * p.v_dim / 4 + 31) / 32 * 32), y = std::max(1, std::min(512 / x, p.H));
  const size_t smem = ((size_t)16 * x * y + (size_t)p.H * p.H + (size_t)p.H * p.splits) * sizeof(float);
  static bool configured[kMaxDevices] = {};
  if (first_call_on_device(configured))
    cuda_check(cudaFuncSetAttribute(talk_mix_slices_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024), "talk_mix smem");
  launch_pdl(talk_mix_slices_kernel<T>, dim3(p.tokens), dim3(x, y), smem, s, p);
  cuda_check(cudaGetLastError(), "talk_mix_slices_kernel");
}
template <typename T>
void launch_mix_rows(const TalkMixParams& p, cudaStream_t s) {
  const int x = std::min(256, (p.G * p.v_dim / 4 + 31) / 32 * 32), y = p.tokens >= 8 * sm_count() ? std::max(1, 256 / x) : 1;
  const size_t smem = ((size_t)p.H * p.H + (size_t)y * p.H) * sizeof(float);
  launch_pdl(talk_mix_rows_kernel<T>, dim3((p.tokens + y - 1) / y), dim3(x, y), smem, s, p);
  cuda_check(cudaGetLastError(), "talk_mix_rows_kernel");
}

template <typename T, int NC>
void launch_mix(const TalkMixParams& p, cudaStream_t s) {
  const size_t smem = ((size_t)p.H * p.splits + (size_t)p.H * NC) * sizeof(float);
  static bool configured[kMaxDevices] = {};
  if (first_call_on_device(configured))
    cuda_check(cudaFuncSetAttribute(talk_mix_kernel<T, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024), "talk_mix smem");
  if (smem > 200 * 1024) throw std::runtime_error("talk_mix: too many heads");
  launch_pdl(talk_mix_kernel<T, NC>, dim3(p.tokens, (p.G * p.v_dim + NC - 1) / NC), dim3(256), smem, s, p);
  cuda_check(cudaGetLastError(), "talk_mix_kernel");
}

// the table of a tile's factors: heads of a group x distances, rows spaced so that the lanes of a warp hit distinct banks
void plan_table(Talk& a) {
  const int n = 127 / a.group + 1 + kTile, shift = (32 + a.group - 1) / a.group % 32;
  a.tab_stride = n + ((shift - n) % 32 + 32) % 32;
  a.tab_entries = a.group * a.tab_stride;
  a.tab_bufs = 2 * a.tab_entries <= kTable ? 2 : 1;
}

template <int DK, int NC>
void launch_decode_cols(const Talk& a, const MapsAttnParams& p, int splits, cudaStream_t s) {
  static bool configured[kMaxDevices] = {};
  if (first_call_on_device(configured))
    cuda_check(cudaFuncSetAttribute(talk_decode_kernel<DK, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, TalkDecode<DK, NC>::kTotal), "talk_decode smem");
  const int col_ctas = a.wv / NC, tiles = (std::min(p.max_q_len, kDecodeRows / a.group) * a.H + 15) / 16;
  launch_pdl(talk_decode_kernel<DK, NC>, dim3(tiles * col_ctas, p.num_seqs, splits), dim3(128), TalkDecode<DK, NC>::kTotal, s, a, col_ctas, splits);
}
template <int DK>
void launch_decode(const Talk& a, const MapsAttnParams& p, int splits, cudaStream_t s) {
  if (a.wv == 64) launch_decode_cols<DK, 64>(a, p, splits, s);
  else if (a.wv % 256 == 0) launch_decode_cols<DK, 256>(a, p, splits, s);
  else launch_decode_cols<DK, 128>(a, p, splits, s);
  cuda_check(cudaGetLastError(), "talk_decode_kernel");
}

// tensor map of a pool of rows of wv values as [64-column part][row][64 values], in boxes of a page's rows and up to kCols columns
CUtensorMap value_map(const void* pool, uint64_t rows, int wv) {
  static std::unordered_map<std::string, CUtensorMap> maps;
  const std::string key = std::to_string(reinterpret_cast<uintptr_t>(pool)) + "/" + std::to_string(rows) + "/" + std::to_string(wv);
  auto it = maps.find(key);
  if (it != maps.end()) return it->second;
  if (maps.size() > 4096) maps.clear();
  return maps.emplace(key, make_tmap_parts(pool, rows, wv, kPage, std::min(kCols, wv) / 64)).first->second;
}

template <int DK>
void launch_prefill(const Talk& a, const MapsAttnParams& p, int min_rows, cudaStream_t s) {
  static bool configured[kMaxDevices] = {};
  if (first_call_on_device(configured))
    cuda_check(cudaFuncSetAttribute(talk_prefill_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, TalkTile<DK>::kTotal), "talk_prefill smem");
  const uint64_t n = (uint64_t)p.num_blocks * a.block_size;
  const CUtensorMap km = pool_map(p.k_cache, n * a.G, DK), vm = value_map(p.v_cache, n, a.wv);
  const int col_ctas = (a.wv + kCols - 1) / kCols;
  const dim3 grid((p.max_q_len * a.group + kRows - 1) / kRows, a.G * col_ctas, p.num_seqs);
  // in plain stream order: a kernel that takes all tensor memory of its SMs neither starts early nor lets others start
  talk_prefill_kernel<DK><<<grid, kThreads, TalkTile<DK>::kTotal, s>>>(km, vm, a, min_rows, col_ctas);
  cuda_check(cudaGetLastError(), "talk_prefill_kernel");
}
}  // namespace

bool attention_spread_tc_supported(int group, int wk, int wv, int block_size, int f32) {
  Talk a{};
  a.group = group;
  plan_table(a);
  return !f32 && (wk == 64 || wk == 128) && (wv == 64 || wv % kPiece == 0) && block_size % kPage == 0 && a.tab_entries <= kTable;
}

// key slices for a step (1 where some sequence runs as a prompt)
int attention_spread_splits(int num_seqs, int max_q_len, int H, int G, int wv, int max_kv_len, int window) {
  if (max_q_len * (H / G) > kDecodeRows) return 1;
  const long long ctas = (long long)num_seqs * ((max_q_len * H + 15) / 16) * ((wv + 255) / 256);
  const int keys = window > 0 ? std::min(max_kv_len, window + max_q_len) : max_kv_len, pages = (keys + kPage - 1) / kPage;
  if (ctas >= sm_count()) return 1;
  return std::max(1, (int)std::min<long long>({2 * sm_count() / ctas, (pages + 7) / 8, 32}));
}

int attention_spread_tc(const MapsAttnParams& p, int splits, int* status, cudaStream_t s) {
  Talk a{};
  a.q = static_cast<const bf16*>(p.q), a.kc = static_cast<const bf16*>(p.k_cache), a.vc = static_cast<const bf16*>(p.v_cache), a.block_tables = p.block_tables, a.max_blocks = p.max_blocks, a.q_starts = p.q_starts, a.positions = p.positions;
  a.H = p.H, a.G = p.G, a.group = p.H / p.G, a.block_size = p.block_size, a.window = p.window, a.wv = p.wv;
  a.scale_log2 = p.scale * kLog2e, a.r1 = p.r1, a.r2 = p.r2, a.part_o = p.part_o, a.part_ml = p.part_ml, a.status = status;
  plan_table(a);
  int launches = 0;
  const bool prompts = p.max_q_len * a.group > kDecodeRows;
  if (prompts && splits != 1) throw std::runtime_error("attention_talk: prompts have one key slice");
  if (p.min_q_len * a.group <= kDecodeRows) {
    if (p.wk == 64) launch_decode<64>(a, p, splits, s);
    else launch_decode<128>(a, p, splits, s);
    ++launches;
  }
  if (prompts) {
    if (p.wk == 64) launch_prefill<64>(a, p, kDecodeRows + 1, s);
    else launch_prefill<128>(a, p, kDecodeRows + 1, s);
    ++launches;
  }
  return launches;
}

void talk_mix(const TalkMixParams& p, cudaStream_t s) {
  if (p.tokens <= 0) return;
  if (p.splits > 32) throw std::runtime_error("talk_mix: at most 32 key slices");
  if (p.v_dim % 4 == 0 && p.H <= 96 && (p.splits > 1 || p.tokens < 2 * sm_count())) {
    if (p.f32) launch_mix_slices<float>(p, s);
    else launch_mix_slices<bf16>(p, s);
    return;
  }
  if (p.v_dim % 4 == 0 && p.H <= 96) {
    TalkMixParams q = p;
    q.vec = p.ldo % 4 == 0 && reinterpret_cast<uintptr_t>(p.out) % (p.f32 ? 16 : 8) == 0;
    if (p.f32) launch_mix_rows<float>(q, s);
    else launch_mix_rows<bf16>(q, s);
    return;
  }
  const bool wide = p.tokens >= 256 && p.H <= 128;
  if (p.f32) wide ? launch_mix<float, 128>(p, s) : launch_mix<float, 32>(p, s);
  else wide ? launch_mix<bf16, 128>(p, s) : launch_mix<bf16, 32>(p, s);
}

}  // namespace fllm
