// Lightning attention on prompts, in matrix form on the tensor cores: per head, with a constant decay d and states S [K][V],
//   S_t = d S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t
// over chunks of 64 tokens (i, j inside the chunk, S in front of it, n its tokens):
//   o_i = d^(i+1) S^T q_i + sum_(j <= i) d^(i-j) (q_i . k_j) v_j
//   S  <- d^n S + sum_j k_j (d^(n-1-j) v_j)^T
// One CTA per (sequence, head, slice of V columns) walks the chunks; the next chunk arrives by cp.async under the products. The
// state stays in registers as fp32 accumulators; for the products it travels as the sum of two bf16 values, like the weights
// d^(i-j) (q_i . k_j); the decayed values of the state's update travel as the sum of three (24 significant bits). q, k and v
// (bf16, activations applied) are exact operands. States and batch layout as in recurrent_ssd.cu (rows [slot][head][V][K]).
#include <algorithm>

#include "attention_util.cuh"
#include "fllm_ops.h"
#include "ptx.cuh"
#include "tma_host.h"

namespace fllm {
namespace {
constexpr int kChunk = 64;

struct ChunkArgs {
  const bf16 *q, *k, *v;
  long long ldq, ldk, ldv, ldo;
  const float* decay;
  float* state;                       // [slots][H][V][K]
  const int *q_starts, *seq_state, *positions;
  bf16* out;
  int H, K, V, min_tokens;            // shorter sequences are left to another path
};

// 16 bytes, zeros where `live` is off
__device__ __forceinline__ void cp_async16_or_zero(void* smem, const void* gmem, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem)), "l"(gmem), "r"(live ? 16 : 0) : "memory");
}

template <int DK, int VS>
struct ChunkTile {
  static constexpr int kLd = VS + 8;                                       // row length of the narrow tiles: rows in distinct banks
  static constexpr int kStage = 2 * kChunk * DK * 2 + kChunk * kLd * 2;    // q, k, v
  static constexpr int kTotal = 2 * kStage + 3 * kChunk * kLd * 2 + 2 * DK * kLd * 2 + (kChunk + 1) * 4 + 16;
};

template <int DK, int VS>
__global__ void __launch_bounds__(128) decay_chunk_kernel(const ChunkArgs a) {
  using L = ChunkTile<DK, VS>;
  constexpr int LD = L::kLd, MT = DK / 64, NT = VS / 8;                    // m tiles of a warp's state rows, n tiles of the slice
  extern __shared__ __align__(128) uint8_t smem[];
  bf16* terms = reinterpret_cast<bf16*>(smem + 2 * L::kStage);             // [3][token][LD] decayed values
  bf16* shi = terms + 3 * kChunk * LD;                                     // [DK][LD] state, leading and second term
  bf16* slo = shi + DK * LD;
  float* power = reinterpret_cast<float*>(slo + DK * LD);                  // d^0 .. d^64
  const int slices = (a.V + VS - 1) / VS;
  const int h = blockIdx.x / slices, v0 = (blockIdx.x % slices) * VS, s = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3, j4 = lane >> 3;
  pdl_wait();
  const int t0 = a.q_starts[s], n = a.q_starts[s + 1] - t0;
  if (n <= 0 || n < a.min_tokens) return;
  if (threadIdx.x <= kChunk) {
    double r = 1.0, b = (double)a.decay[h];
    for (int e = threadIdx.x; e; e >>= 1) {
      if (e & 1) r *= b;
      b *= b;
    }
    power[threadIdx.x] = (float)r;
  }
  const bf16* q = a.q + (long long)t0 * a.ldq + (long long)h * a.K;
  const bf16* k = a.k + (long long)t0 * a.ldk + (long long)h * a.K;
  const bf16* v = a.v + (long long)t0 * a.ldv + (long long)h * a.V + v0;
  auto fetch = [&](int c) {
    bf16* qs = reinterpret_cast<bf16*>(smem + (c & 1) * L::kStage);
    bf16 *ks = qs + kChunk * DK, *vs = ks + kChunk * DK;
    const int base = c * kChunk;
    for (int i = threadIdx.x; i < kChunk * (DK / 8); i += 128) {
      const int r = i / (DK / 8), p = i % (DK / 8);
      const bool live = base + r < n && p * 8 < a.K;
      const long long t = live ? base + r : 0;
      const int col = live ? p * 8 : 0;
      cp_async16_or_zero(tile_ptr<DK>(qs, r, p), q + t * a.ldq + col, live);
      cp_async16_or_zero(tile_ptr<DK>(ks, r, p), k + t * a.ldk + col, live);
    }
    for (int i = threadIdx.x; i < kChunk * (VS / 8); i += 128) {
      const int r = i / (VS / 8), p = i % (VS / 8);
      const bool live = base + r < n && v0 + p * 8 < a.V;
      cp_async16_or_zero(vs + r * LD + p * 8, v + (live ? (long long)(base + r) * a.ldv + p * 8 : 0), live);
    }
    cp_async_commit();
  };
  fetch(0);
  float S[MT][NT][4];                                                      // state rows warp * DK / 4 + 16 m + g (+ 8), columns 8 n + 2 t4 (+ 1)
  float* st = a.state + ((long long)a.seq_state[s] * a.H + h) * a.V * a.K;
  const bool fresh = a.positions[t0] == 0;
  auto each = [&](auto f) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) f(S[m][nt][e], warp * (DK / 4) + 16 * m + g + 8 * (e >> 1), v0 + 8 * nt + 2 * t4 + (e & 1));
  };
  each([&](float& x, int row, int col) { x = !fresh && row < a.K && col < a.V ? st[(long long)col * a.K + row] : 0.f; });

  const int chunks = (n + kChunk - 1) / kChunk;
  for (int c = 0; c < chunks; ++c) {
    const int cnt = min(kChunk, n - c * kChunk);
    if (c + 1 < chunks) {
      fetch(c + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    bf16* qs = reinterpret_cast<bf16*>(smem + (c & 1) * L::kStage);
    bf16 *ks = qs + kChunk * DK, *vs = ks + kChunk * DK;
    // ---- the state in two terms, the decayed values in three
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int at = (warp * (DK / 4) + 16 * m + g + 8 * i) * LD + 8 * nt + 2 * t4;
          const uint32_t hi = pack_bf16x2(S[m][nt][2 * i], S[m][nt][2 * i + 1]);
          const float2 back = unpack_bf16x2(hi);
          *reinterpret_cast<uint32_t*>(shi + at) = hi;
          *reinterpret_cast<uint32_t*>(slo + at) = pack_bf16x2(S[m][nt][2 * i] - back.x, S[m][nt][2 * i + 1] - back.y);
        }
    for (int i = threadIdx.x; i < kChunk * (VS / 2); i += 128) {
      const int r = i / (VS / 2), at = r * LD + 2 * (i % (VS / 2));
      const float w = r < cnt ? power[cnt - 1 - r] : 0.f;
      float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(vs + at));
      x.x *= w, x.y *= w;
#pragma unroll
      for (int term = 0; term < 3; ++term) {
        const uint32_t b = pack_bf16x2(x.x, x.y);
        const float2 back = unpack_bf16x2(b);
        *reinterpret_cast<uint32_t*>(terms + term * kChunk * LD + at) = b;
        x.x -= back.x, x.y -= back.y;
      }
    }
    __syncthreads();
    // ---- outputs: 16 tokens per warp
    const int row0 = warp * 16;
    if (row0 < cnt) {
      uint32_t qf[DK / 16][4];
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) ldsm_x4(qf[kk], tile_ptr<DK>(qs, row0 + (lane & 15), 2 * kk + (lane >> 4)));
      float o[NT][4];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk)
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t b[4];
          const int at = (kk * 16 + (j4 & 1) * 8 + (lane & 7)) * LD + 8 * (nt + (j4 >> 1));
          ldsm_x4_t(b, shi + at);
          mma_bf16(o[nt], qf[kk], b[0], b[1]);
          mma_bf16(o[nt + 1], qf[kk], b[2], b[3]);
          ldsm_x4_t(b, slo + at);
          mma_bf16(o[nt], qf[kk], b[0], b[1]);
          mma_bf16(o[nt + 1], qf[kk], b[2], b[3]);
        }
      const float d0 = power[row0 + g + 1], d1 = power[row0 + g + 9];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) o[nt][0] *= d0, o[nt][1] *= d0, o[nt][2] *= d1, o[nt][3] *= d1;
      for (int ct = 0; ct <= warp; ++ct) {                                 // 16 earlier tokens at a time
        float x[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) x[i][0] = x[i][1] = x[i][2] = x[i][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          uint32_t b[4];
          ldsm_x4(b, tile_ptr<DK>(ks, ct * 16 + (j4 >> 1) * 8 + (lane & 7), 2 * kk + (j4 & 1)));
          mma_bf16(x[0], qf[kk], b[0], b[1]);
          mma_bf16(x[1], qf[kk], b[2], b[3]);
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int back = row0 + g + 8 * i - (ct * 16 + nb * 8 + 2 * t4);       // how far the first of the two tokens lies behind
            const float p0 = back >= 0 ? x[nb][2 * i] * power[back] : 0.f, p1 = back >= 1 ? x[nb][2 * i + 1] * power[back - 1] : 0.f;
            const uint32_t hi = pack_bf16x2(p0, p1);
            const float2 f = unpack_bf16x2(hi);
            ph[nb * 2 + i] = hi;
            pl[nb * 2 + i] = pack_bf16x2(p0 - f.x, p1 - f.y);
          }
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t b[4];
          ldsm_x4_t(b, vs + (ct * 16 + (j4 & 1) * 8 + (lane & 7)) * LD + 8 * (nt + (j4 >> 1)));
          mma_bf16(o[nt], ph, b[0], b[1]);
          mma_bf16(o[nt + 1], ph, b[2], b[3]);
          mma_bf16(o[nt], pl, b[0], b[1]);
          mma_bf16(o[nt + 1], pl, b[2], b[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = row0 + g + 8 * i;
        if (r >= cnt) continue;
        bf16* dst = a.out + (long long)(t0 + c * kChunk + r) * a.ldo + (long long)h * a.V;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const int col = v0 + 8 * nt + 2 * t4;                            // (V is even)
          if (col < a.V) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16x2(o[nt][2 * i], o[nt][2 * i + 1]);
        }
      }
    }
    // ---- state: DK / 4 rows per warp
    const float whole = power[cnt];
    each([&](float& x, int, int) { x *= whole; });
    for (int kt = 0; kt < (cnt + 15) / 16; ++kt) {
      uint32_t af[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
        ldsm_x4_t(af[m], tile_ptr<DK>(ks, kt * 16 + (lane >> 4) * 8 + (lane & 7), (warp * (DK / 4) + 16 * m) / 8 + (j4 & 1)));
#pragma unroll
      for (int term = 0; term < 3; ++term)
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t b[4];
          ldsm_x4_t(b, terms + (term * kChunk + kt * 16 + (j4 & 1) * 8 + (lane & 7)) * LD + 8 * (nt + (j4 >> 1)));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(S[m][nt], af[m], b[0], b[1]);
            mma_bf16(S[m][nt + 1], af[m], b[2], b[3]);
          }
        }
    }
    __syncthreads();                                                       // the chunk's buffer and the shared terms are free
  }
  each([&](float& x, int row, int col) {
    if (row < a.K && col < a.V) st[(long long)col * a.K + row] = x;
  });
}

template <int DK, int VS>
void launch_chunk(const ChunkArgs& a, int B, cudaStream_t s) {
  using L = ChunkTile<DK, VS>;
  static bool configured[kMaxDevices] = {};
  if (first_call_on_device(configured))
    cuda_check(cudaFuncSetAttribute(decay_chunk_kernel<DK, VS>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::kTotal), "decay_chunk smem");
  launch_pdl(decay_chunk_kernel<DK, VS>, dim3(a.H * ((a.V + VS - 1) / VS), B), dim3(128), L::kTotal, s, a);
}
}  // namespace

bool decay_chunk_supported(int K, int V) { return K % 8 == 0 && V % 8 == 0 && K <= 128; }

int decay_chunk(const SsdScanParams& p, int min_tokens, cudaStream_t s) {
  if (p.B <= 0) return 0;
  if (p.f32 || !decay_chunk_supported(p.N, p.P) || p.G != p.H) return -1;
  const uintptr_t any = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.Bm) | reinterpret_cast<uintptr_t>(p.Cm);
  if (any % 16 || p.ldx % 8 || p.ldb % 8 || p.ldc % 8 || p.ldy % 2 || reinterpret_cast<uintptr_t>(p.y) % 4) return -2;
  const ChunkArgs a{static_cast<const bf16*>(p.Cm), static_cast<const bf16*>(p.Bm), static_cast<const bf16*>(p.x), p.ldc, p.ldb, p.ldx, p.ldy, p.A,
                    p.state, p.q_starts, p.seq_state, p.positions, static_cast<bf16*>(p.y), p.H, p.N, p.P, min_tokens};
  // narrower slices (more CTAs, each with the chunk's scores to itself) as long as two CTAs per SM hold them all
  const int longest = std::max(p.max_q_len, 1), walks = std::min(p.B, (p.tokens + longest - 1) / longest);      // about as many as run that long
  const bool narrow = (long long)p.H * ((p.P + 15) / 16) * walks <= 2 * sm_count();
  if (p.N <= 64) narrow ? launch_chunk<64, 16>(a, p.B, s) : launch_chunk<64, 32>(a, p.B, s);
  else narrow ? launch_chunk<128, 16>(a, p.B, s) : launch_chunk<128, 32>(a, p.B, s);
  cuda_check(cudaGetLastError(), "decay_chunk_kernel");
  return 0;
}

}  // namespace fllm
