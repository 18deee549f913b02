// The Mamba-2 recurrence (one decay, one step size per head) with any head and state width, in bf16 and fp32:
//   dt = clamp(softplus(dt_raw + bias));  S[p][n] <- exp(dt A) S[p][n] + dt x[p] B[n];  y[p] = sum_n S[p][n] C[n] + D x[p]
// Batch layout and states as in recurrent.cu (state rows [slot][head][P][N] in fp32); all arithmetic is fp32.
//
// ssd_scan_kernel walks a sequence's tokens, one CTA per (sequence, head, slice of state rows). TPK lanes share RPT rows, lane l
// holding the columns 4 (l + TPK j) + 0..3 of each as pairs for the packed fp32 instructions. Tokens come in chunks: eight
// threads per token fetch B and C one chunk ahead in their stored form and leave them in shared memory as fp32 with the
// token's decay and step size, so the walk over a chunk touches shared memory and registers only. A token's columns are
// independent, so the walk is bound by the rate of its fp32 instructions, not by a chain.
//
// ssd_decode_kernel serves steps of single tokens: inputs straight from global memory, no shared memory, many CTAs that keep
// state reads in flight (a decoded token reads and writes the whole state once).
//
// NP: state columns in registers; EXACT: the state width is NP and rows are 16-byte aligned, otherwise it is N <= NP and rows
// are read value by value.
#include "fllm_ops.h"
#include "recurrent_util.cuh"

namespace fllm {
namespace {

constexpr int kSsdChunk = 16;

// pairs of fp32 values in one 64-bit register
__device__ __forceinline__ uint64_t pair(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpair(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
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

template <typename T>
struct SsdArgs {
  const T *x, *dt, *Bm, *Cm;
  long long ldx, lddt, ldb, ldc, ldy;
  const float *A, *D, *dt_bias;
  float* state;                       // [slots][H][P][N]
  const int *q_starts, *seq_state, *positions;
  T* y;
  int H, P, G, N;
  float dt_min, dt_max;
  int skip_from;                      // sequences with at least this many tokens in the step are left to another path (0 = none)
};

template <typename T, int NP, bool EXACT, int RPT>
__global__ void __launch_bounds__(128) ssd_scan_kernel(const SsdArgs<T> a) {
  constexpr int NPT = 16, TPK = NP / NPT, RG = 128 / TPK, ROWS = RPT * RG, C = kSsdChunk, EPT = NP / 8, VPT = ROWS * C / 128;
  __shared__ __align__(16) float sb[C][NP], sc[C][NP];
  __shared__ float sx[C][ROWS];
  __shared__ float2 sg[C];                               // decay, step size
  const int N = EXACT ? NP : a.N;
  const int ptiles = (a.P + ROWS - 1) / ROWS;
  const int h = blockIdx.x / ptiles, p0 = (blockIdx.x % ptiles) * ROWS, row = threadIdx.x / TPK;      // rows p0 + row + RG r
  const int lk = threadIdx.x % TPK, s = blockIdx.y;
  const int t0 = a.q_starts[s], n = a.q_starts[s + 1] - t0;
  if (n <= 0 || (a.skip_from > 0 && n >= a.skip_from)) return;
  float* st = a.state + ((long long)a.seq_state[s] * a.H + h) * a.P * N;
  const bool fresh = a.positions[t0] == 0;
  uint64_t S[RPT][NPT / 2];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    float v[NPT];
#pragma unroll
    for (int i = 0; i < NPT; ++i) v[i] = 0.f;
    if (!fresh) load_state<TPK, EXACT>(st + (long long)min(p0 + row + RG * r, a.P - 1) * N, lk, N, v);
#pragma unroll
    for (int i = 0; i < NPT / 2; ++i) S[r][i] = pair(v[2 * i], v[2 * i + 1]);
  }
  const float A = a.A[h], D = a.D != nullptr ? a.D[h] : 0.f, dtb = a.dt_bias != nullptr ? a.dt_bias[h] : 0.f;
  // fetching: thread = (token tt of the chunk, share part of its rows); shares are groups of eight values, so that the
  // shared-memory stores of a token's eight threads spread over the banks
  constexpr bool WIDE = EXACT && EPT % 8 == 0;
  constexpr int WORDS = WIDE ? EPT * (int)sizeof(T) / 16 : 1, LOOSE = WIDE ? 1 : EPT, PER8 = (int)sizeof(T) / 2;      // 16-byte words per group
  const int tt = threadIdx.x / 8, part = threadIdx.x % 8;
  const long long go = (long long)(h / (a.H / a.G)) * N;
  auto column = [&](int i) { return EPT % 8 == 0 ? 8 * (part + 8 * (i / 8)) + i % 8 : part * EPT + i; };
  uint4 bw[WORDS], cw[WORDS];
  float bl[LOOSE], cl[LOOSE];
  T xr[VPT], dr{};
  auto fetch = [&](int base) {
    const int left = n - base;
    if (tt < left) {
      const long long t = t0 + base + tt;
      const T *bp = a.Bm + t * a.ldb + go, *cp = a.Cm + t * a.ldc + go;
      if constexpr (WIDE) {
#pragma unroll
        for (int i = 0; i < WORDS; ++i) {
          const int c = 8 * (part + 8 * (i / PER8)) + (i % PER8) * (16 / (int)sizeof(T));
          bw[i] = *reinterpret_cast<const uint4*>(bp + c);
          cw[i] = *reinterpret_cast<const uint4*>(cp + c);
        }
      } else {
#pragma unroll
        for (int i = 0; i < EPT; ++i) {
          const int c = column(i);
          bl[i] = c < N ? ld1(bp + c) : 0.f;
          cl[i] = c < N ? ld1(cp + c) : 0.f;
        }
      }
      if (part == 0) dr = a.dt[t * a.lddt + h];
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int e = threadIdx.x + i * 128, tv = e / ROWS, rv = min(p0 + e % ROWS, a.P - 1);
      if (tv < left) xr[i] = a.x[(t0 + base + tv) * a.ldx + (long long)h * a.P + rv];
    }
  };
  fetch(0);
  for (int base = 0; base < n; base += C) {
    const int cnt = min(C, n - base);
    __syncthreads();                                     // the chunk before is consumed
    if (tt < cnt) {
      float br[EPT], cr[EPT];
      if constexpr (WIDE) {
        const T *bt = reinterpret_cast<const T*>(bw), *ct = reinterpret_cast<const T*>(cw);
#pragma unroll
        for (int i = 0; i < EPT; ++i) br[i] = ld1(bt + i), cr[i] = ld1(ct + i);
      } else {
#pragma unroll
        for (int i = 0; i < EPT; ++i) br[i] = bl[i], cr[i] = cl[i];
      }
      if constexpr (EPT % 4 == 0) {
#pragma unroll
        for (int i = 0; i < EPT; i += 4) {
          *reinterpret_cast<float4*>(&sb[tt][column(i)]) = make_float4(br[i], br[i + 1], br[i + 2], br[i + 3]);
          *reinterpret_cast<float4*>(&sc[tt][column(i)]) = make_float4(cr[i], cr[i + 1], cr[i + 2], cr[i + 3]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < EPT; ++i) sb[tt][column(i)] = br[i], sc[tt][column(i)] = cr[i];
      }
      if (part == 0) {
        const float dt = fminf(fmaxf(softplus_t<T>(ld1(&dr) + dtb), a.dt_min), a.dt_max);
        sg[tt] = make_float2(exp_t<T>(dt * A), dt);
      }
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int e = threadIdx.x + i * 128;
      if (e / ROWS < cnt) sx[e / ROWS][e % ROWS] = ld1(&xr[i]);
    }
    __syncthreads();
    if (base + C < n) fetch(base + C);
    T* yp = a.y + (long long)(t0 + base) * a.ldy + (long long)h * a.P + p0 + row;
#pragma unroll 2
    for (int i = 0; i < cnt; ++i, yp += a.ldy) {
      uint64_t b2[NPT / 2], c2[NPT / 2];
#pragma unroll
      for (int j = 0; j < NPT / 4; ++j) {
        const ulonglong2 bv = *reinterpret_cast<const ulonglong2*>(&sb[i][4 * (lk + TPK * j)]);
        const ulonglong2 cv = *reinterpret_cast<const ulonglong2*>(&sc[i][4 * (lk + TPK * j)]);
        b2[2 * j] = bv.x, b2[2 * j + 1] = bv.y, c2[2 * j] = cv.x, c2[2 * j + 1] = cv.y;
      }
      const float2 g = sg[i];
      const uint64_t d2 = pair(g.x, g.x);
#pragma unroll
      for (int r = 0; r < RPT; ++r) {
        const float xv = sx[i][row + RG * r], u = g.y * xv;
        const uint64_t u2 = pair(u, u);
        uint64_t o2[2] = {0, 0};                           // two chains of packed sums
#pragma unroll
        for (int j = 0; j < NPT / 2; ++j) {
          S[r][j] = fma2(b2[j], u2, mul2(S[r][j], d2));
          o2[j & 1] = fma2(S[r][j], c2[j], o2[j & 1]);
        }
        const float2 e = unpair(o2[0]), f = unpair(o2[1]);
        const float o = row_sum<TPK>((e.x + e.y) + (f.x + f.y));
        if (lk == 0 && p0 + row + RG * r < a.P) st1(yp + RG * r, fmaf(D, xv, o));
      }
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    if (p0 + row + RG * r >= a.P) continue;
    float v[NPT];
#pragma unroll
    for (int i = 0; i < NPT / 2; ++i) {
      const float2 f = unpair(S[r][i]);
      v[2 * i] = f.x, v[2 * i + 1] = f.y;
    }
    store_state<TPK, EXACT>(st + (long long)(p0 + row + RG * r) * N, lk, N, v);
  }
}

template <typename T, int NP, bool EXACT, int RPT>
__global__ void __launch_bounds__(128) ssd_decode_kernel(const SsdArgs<T> a) {
  constexpr int NPT = 16, TPK = NP / NPT, RG = 128 / TPK, ROWS = RPT * RG;
  const int N = EXACT ? NP : a.N;
  const int ptiles = (a.P + ROWS - 1) / ROWS;
  const int h = blockIdx.x / ptiles, p0 = (blockIdx.x % ptiles) * ROWS + threadIdx.x / TPK;      // rows p0 + RG r
  const int lk = threadIdx.x % TPK, s = blockIdx.y;
  const int t0 = a.q_starts[s], n = a.q_starts[s + 1] - t0;
  if (n <= 0 || (a.skip_from > 0 && n >= a.skip_from)) return;
  float* st = a.state + ((long long)a.seq_state[s] * a.H + h) * a.P * N;
  float S[RPT][NPT];
  const bool fresh = a.positions[t0] == 0;
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
#pragma unroll
    for (int i = 0; i < NPT; ++i) S[r][i] = 0.f;
    if (!fresh) load_state<TPK, EXACT>(st + (long long)min(p0 + RG * r, a.P - 1) * N, lk, N, S[r]);
  }
  const float A = a.A[h], D = a.D != nullptr ? a.D[h] : 0.f, dtb = a.dt_bias != nullptr ? a.dt_bias[h] : 0.f;
  const long long go = (long long)(h / (a.H / a.G)) * N;
  for (long long t = t0; t < t0 + n; ++t) {
    const T *bp = a.Bm + t * a.ldb + go, *cp = a.Cm + t * a.ldc + go;
    float B[NPT], C[NPT];
#pragma unroll
    for (int j = 0; j < NPT / 4; ++j) {
      const int c = 4 * (lk + TPK * j);
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        float2 b2 = make_float2(0.f, 0.f), c2 = b2;
        if (EXACT) {
          b2 = ld2(bp + c + e), c2 = ld2(cp + c + e);
        } else {
          if (c + e < N) b2.x = ld1(bp + c + e), c2.x = ld1(cp + c + e);
          if (c + e + 1 < N) b2.y = ld1(bp + c + e + 1), c2.y = ld1(cp + c + e + 1);
        }
        B[4 * j + e] = b2.x, B[4 * j + e + 1] = b2.y, C[4 * j + e] = c2.x, C[4 * j + e + 1] = c2.y;
      }
    }
    const float dt = fminf(fmaxf(softplus_t<T>(ld1(a.dt + t * a.lddt + h) + dtb), a.dt_min), a.dt_max);
    const float d = exp_t<T>(dt * A);
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int p = p0 + RG * r;
      const float xv = ld1(a.x + t * a.ldx + (long long)h * a.P + min(p, a.P - 1)), u = dt * xv;
      float o[2] = {0.f, 0.f};
#pragma unroll
      for (int i = 0; i < NPT; ++i) {
        S[r][i] = fmaf(B[i], u, d * S[r][i]);
        o[i & 1] = fmaf(S[r][i], C[i], o[i & 1]);
      }
      const float tot = row_sum<TPK>(o[0] + o[1]);
      if (lk == 0 && p < a.P) st1(a.y + t * a.ldy + (long long)h * a.P + p, fmaf(D, xv, tot));
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r)
    if (p0 + RG * r < a.P) store_state<TPK, EXACT>(st + (long long)(p0 + RG * r) * N, lk, N, S[r]);
}
}  // namespace

int ssd_scan(const SsdScanParams& p, cudaStream_t stream) {
  if (p.B <= 0) return 0;
  if (p.G <= 0 || p.H % p.G || p.N <= 0 || p.P <= 0) return -1;
  if (p.N > 256) return -2;
  const int unit = p.f32 ? 4 : 8;
  const bool exact = (p.N == 16 || p.N == 32 || p.N == 64 || p.N == 128 || p.N == 256) && aligned16(p.Bm) && aligned16(p.Cm) && p.ldb % unit == 0 && p.ldc % unit == 0;
  auto args = [&](auto zero) {
    using T = decltype(zero);
    return SsdArgs<T>{static_cast<const T*>(p.x), static_cast<const T*>(p.dt), static_cast<const T*>(p.Bm), static_cast<const T*>(p.Cm),
                      p.ldx, p.lddt, p.ldb, p.ldc, p.ldy, p.A, p.D, p.dt_bias, p.state, p.q_starts, p.seq_state, p.positions,
                      static_cast<T*>(p.y), p.H, p.P, p.G, p.N, p.dt_min, p.dt_max, p.skip_from};
  };
#define FLLM_SSD(T_, NP_, EXACT_)                                                                                     \
  {                                                                                                                   \
    constexpr int rows = 128 / (NP_ / 16);                                                                            \
    if (p.tokens == p.B)                                                                                              \
      ssd_decode_kernel<T_, NP_, EXACT_, 1><<<dim3(p.H * ((p.P + rows - 1) / rows), p.B), 128, 0, stream>>>(args(T_{}));             \
    else                                                                                                              \
      ssd_scan_kernel<T_, NP_, EXACT_, 2><<<dim3(p.H * ((p.P + 2 * rows - 1) / (2 * rows)), p.B), 128, 0, stream>>>(args(T_{}));     \
    return 0;                                                                                                         \
  }
#define FLLM_SSD_N(T_, EXACT_)                    \
  {                                               \
    if (p.N <= 16) FLLM_SSD(T_, 16, EXACT_)       \
    if (p.N <= 32) FLLM_SSD(T_, 32, EXACT_)       \
    if (p.N <= 64) FLLM_SSD(T_, 64, EXACT_)       \
    if (p.N <= 128) FLLM_SSD(T_, 128, EXACT_)     \
    FLLM_SSD(T_, 256, EXACT_)                     \
  }
  if (p.f32) {
    if (exact) FLLM_SSD_N(float, true)
    FLLM_SSD_N(float, false)
  }
  if (exact) FLLM_SSD_N(bf16, true)
  FLLM_SSD_N(bf16, false)
#undef FLLM_SSD_N
#undef FLLM_SSD
}

}  // namespace fllm
