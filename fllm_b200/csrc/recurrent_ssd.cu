// The Mamba-2 recurrence (one decay, one step size per head) with any head and state width, in bf16 and fp32:
//   dt = clamp(softplus(dt_raw + bias));  S[p][n] <- exp(dt A) S[p][n] + dt x[p] B[n];  y[p] = sum_n S[p][n] C[n] + D x[p]
// Batch layout and states as in recurrent.cu (state rows [slot][head][P][N] in fp32); all arithmetic is fp32.
//
// ssd_scan_kernel walks a sequence's tokens, one CTA per (sequence, head, slice of state rows). TPK lanes share RPT rows, lane l
// holding the columns 4 (l + TPK j) + 0..3 of each as pairs for the packed fp32 instructions. Tokens come in chunks: eight
// threads per token fetch B and C one chunk ahead in their stored form and leave them in shared memory as fp32 with the
// token's decay and step size, so the walk over a chunk touches shared memory and registers only. Four rows per thread keep the
// shared-memory reads below the arithmetic (two where four would leave half the SMs idle). The outputs of four tokens are
// summed over the lanes together, each exchange halving the values a lane carries, so that no sum is computed twice. Inside
// such a group the state is kept over the product of the decays so far (S = P_t S', S' += (dt / P_t) x B, y = P_t S' C): one
// multiplication by the group's whole decay replaces four. Groups that decay too far for that (P below kMinDecay) multiply
// token by token.
//
// ssd_decode_kernel serves steps of single tokens: inputs straight from global memory, no shared memory, many CTAs that keep
// state reads in flight (a decoded token reads and writes the whole state once).
//
// LIN: lightning attention, the same recurrence with a constant decay per head (A holds it), step size 1 and silu on all three
// inputs: S[p][n] <- d S[p][n] + silu(x[p]) silu(B[n]), y[p] = sum_n S[p][n] silu(C[n]).
//
// NP: state columns in registers; EXACT: the state width is NP and rows are 16-byte aligned, otherwise it is N <= NP and rows
// are read value by value.
#include <type_traits>

#include "fllm_ops.h"
#include "ptx.cuh"
#include "recurrent_util.cuh"
#include "tma_host.h"

namespace fllm {
namespace {

constexpr int kSsdChunk = 16;
constexpr float kMinDecay = 2e-9f;           // e^-20: the rounding of the exponents stays at 2e-6

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

// sums over the L lanes of a row group of V values per lane: afterwards v[i] of lane l is the sum of value (l >> rest) * left + i
template <int L, int V>
struct LaneSums {
  static constexpr int left(int l, int v) { return l > 1 && v > 1 ? left(l / 2, v / 2) : v; }
  static constexpr int rest(int l, int v) { return l > 1 && v > 1 ? rest(l / 2, v / 2) : (l > 1 ? 1 + rest(l / 2, v) : 0); }
  static constexpr int kLeft = left(L, V), kRest = rest(L, V);
};
template <int L, int V, int SIZE>
__device__ __forceinline__ void lane_sums(float (&v)[SIZE], int lane) {
  if constexpr (L > 1 && V > 1) {
    const bool upper = (lane & (L / 2)) != 0;
#pragma unroll
    for (int i = 0; i < V / 2; ++i) {
      const float send = upper ? v[i] : v[i + V / 2], keep = upper ? v[i + V / 2] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, L / 2);
    }
    lane_sums<L / 2, V / 2>(v, lane);
  } else if constexpr (L > 1) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
  }
}

template <int NP, int RPT>
struct SsdTile {
  static constexpr int NPT = NP <= 32 ? 4 : 8, TPK = NP / NPT, RG = 128 / TPK, ROWS = RPT * RG, GROUP = 4;
};

template <typename T, int NP, bool EXACT, int RPT, bool LIN>
__global__ void __launch_bounds__(128) ssd_scan_kernel(const SsdArgs<T> a) {
  pdl_wait();
  using L = SsdTile<NP, RPT>;
  constexpr int NPT = L::NPT, TPK = L::TPK, ROWS = L::ROWS, GROUP = L::GROUP, C = kSsdChunk, EPT = NP / 8, VPT = ROWS * C / 128;
  __shared__ __align__(16) float sb[C][NP], sc[C][NP], sx[C][ROWS];
  __shared__ float4 sg[C];                               // P, dt / P, decay, dt
  const int N = EXACT ? NP : a.N;
  const int ptiles = (a.P + ROWS - 1) / ROWS;
  const int h = blockIdx.x / ptiles, p0 = (blockIdx.x % ptiles) * ROWS, row = threadIdx.x / TPK * RPT;      // rows p0 + row + r
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
    if (!fresh) load_state<TPK, EXACT>(st + (long long)min(p0 + row + r, a.P - 1) * N, lk, N, v);
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
      if constexpr (!LIN) dr = a.dt[t * a.lddt + h];
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
    {
      // tokens past the end are steps that change nothing: decay 1, step size 0, zero inputs
      const bool live = tt < cnt;
      float br[EPT], cr[EPT];
      if constexpr (WIDE) {
        const T *bt = reinterpret_cast<const T*>(bw), *ct = reinterpret_cast<const T*>(cw);
#pragma unroll
        for (int i = 0; i < EPT; ++i) br[i] = live ? ld1(bt + i) : 0.f, cr[i] = live ? ld1(ct + i) : 0.f;
      } else {
#pragma unroll
        for (int i = 0; i < EPT; ++i) br[i] = live ? bl[i] : 0.f, cr[i] = live ? cl[i] : 0.f;
      }
      if constexpr (LIN) {
#pragma unroll
        for (int i = 0; i < EPT; ++i) br[i] = silu_t<T>(br[i]), cr[i] = silu_t<T>(cr[i]);
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
      // a warp holds the four tokens of a group: running sum of the exponents over them
      static_assert(GROUP == 4, "eight threads per token");
      if constexpr (LIN) {
        const int n_live = min(tt % 4 + 1, cnt - tt / 4 * 4);      // of the group's tokens up to this one (0 or less: none)
        const float p2 = A * A, P = n_live >= 4 ? p2 * p2 : n_live == 3 ? p2 * A : n_live == 2 ? p2 : n_live == 1 ? A : 1.f;
        if (part == 0) sg[tt] = make_float4(P, live ? 1.f / P : 0.f, live ? A : 1.f, live ? 1.f : 0.f);
      } else {
      const float dt = live ? fminf(fmaxf(softplus_t<T>(ld1(&dr) + dtb), a.dt_min), a.dt_max) : 0.f, e = dt * A;
      float c = e;
      const float c1 = __shfl_up_sync(0xffffffffu, c, 8);
      if (tt % 4 >= 1) c += c1;
      const float c2 = __shfl_up_sync(0xffffffffu, c, 16);
      if (tt % 4 >= 2) c += c2;
      if (part == 0) sg[tt] = make_float4(exp_t<T>(c), dt * exp_t<T>(-c), exp_t<T>(e), dt);
      }
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int e = threadIdx.x + i * 128;
      const float v = e / ROWS < cnt ? ld1(&xr[i]) : 0.f;
      sx[e / ROWS][e % ROWS] = LIN ? silu_t<T>(v) : v;
    }
    __syncthreads();
    if (base + C < n) fetch(base + C);
    for (int i0 = 0; i0 < cnt; i0 += GROUP) {
      float o[GROUP * RPT];
      auto walk = [&](auto scaled) {
        constexpr bool SCALED = decltype(scaled)::value;
#pragma unroll
        for (int k = 0; k < GROUP; ++k) {
          const int i = i0 + k;
          uint64_t b2[NPT / 2], c2[NPT / 2];
#pragma unroll
          for (int j = 0; j < NPT / 4; ++j) {
            const ulonglong2 bv = *reinterpret_cast<const ulonglong2*>(&sb[i][4 * (lk + TPK * j)]);
            const ulonglong2 cv = *reinterpret_cast<const ulonglong2*>(&sc[i][4 * (lk + TPK * j)]);
            b2[2 * j] = bv.x, b2[2 * j + 1] = bv.y, c2[2 * j] = cv.x, c2[2 * j + 1] = cv.y;
          }
          const float4 g = sg[i];
          float xs[RPT];
          if constexpr (RPT == 4) {
            const float4 v = *reinterpret_cast<const float4*>(&sx[i][row]);
            xs[0] = v.x, xs[1] = v.y, xs[2] = v.z, xs[3] = v.w;
          } else {
            const float2 v = *reinterpret_cast<const float2*>(&sx[i][row]);
            xs[0] = v.x, xs[1] = v.y;
          }
          const uint64_t d2 = pair(g.z, g.z);
#pragma unroll
          for (int r = 0; r < RPT; ++r) {
            const float u = (SCALED ? g.y : g.w) * xs[r];
            const uint64_t u2 = pair(u, u);
            uint64_t o2 = 0;
#pragma unroll
            for (int j = 0; j < NPT / 2; ++j) {
              S[r][j] = fma2(b2[j], u2, SCALED ? S[r][j] : mul2(S[r][j], d2));
              o2 = fma2(S[r][j], c2[j], o2);
            }
            const float2 e = unpair(o2);
            o[k * RPT + r] = SCALED ? g.x * (e.x + e.y) : e.x + e.y;
          }
        }
      };
      const float whole = sg[i0 + GROUP - 1].x;
      if (whole > kMinDecay) {
        walk(std::true_type{});
        const uint64_t w2 = pair(whole, whole);
#pragma unroll
        for (int r = 0; r < RPT; ++r)
#pragma unroll
          for (int j = 0; j < NPT / 2; ++j) S[r][j] = mul2(S[r][j], w2);
      } else {
        walk(std::false_type{});
      }
      using Sums = LaneSums<TPK, GROUP * RPT>;
      lane_sums<TPK, GROUP * RPT>(o, lk);
      if (Sums::kRest == 0 || (lk & ((1 << Sums::kRest) - 1)) == 0) {
#pragma unroll
        for (int v = 0; v < Sums::kLeft; ++v) {
          const int at = (lk >> Sums::kRest) * Sums::kLeft + v, i = i0 + at / RPT, p = row + at % RPT;
          if (i < cnt && p0 + p < a.P) st1(a.y + (long long)(t0 + base + i) * a.ldy + (long long)h * a.P + p0 + p, fmaf(D, sx[i][p], o[v]));
        }
      }
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    if (p0 + row + r >= a.P) continue;
    float v[NPT];
#pragma unroll
    for (int i = 0; i < NPT / 2; ++i) {
      const float2 f = unpair(S[r][i]);
      v[2 * i] = f.x, v[2 * i + 1] = f.y;
    }
    store_state<TPK, EXACT>(st + (long long)(p0 + row + r) * N, lk, N, v);
  }
}

// RPT: state rows per thread
template <typename T, int NP, bool EXACT, bool LIN, int RPT>
__global__ void __launch_bounds__(128) ssd_decode_kernel(const SsdArgs<T> a) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int NPT = 16, TPK = NP / NPT, RG = 128 / TPK, ROWS = RPT * RG;
  const int N = EXACT ? NP : a.N;
  const int ptiles = (a.P + ROWS - 1) / ROWS;
  const int h = blockIdx.x / ptiles, p0 = (blockIdx.x % ptiles) * ROWS + threadIdx.x / TPK;      // rows p0 + RG r
  const int lk = threadIdx.x % TPK, s = blockIdx.y;
  const int t0 = a.q_starts[s], n = a.q_starts[s + 1] - t0;
  if (n <= 0 || (a.skip_from > 0 && n >= a.skip_from)) return;
  float* st = a.state + ((long long)a.seq_state[s] * a.H + h) * a.P * N;
  auto row = [&](int r) { return min(p0 + RG * r, a.P - 1); };
  float S[RPT][NPT];
#pragma unroll
  for (int r = 0; r < RPT; ++r)
#pragma unroll
    for (int i = 0; i < NPT; ++i) S[r][i] = 0.f;
  if (a.positions[t0] != 0) {
#pragma unroll
    for (int r = 0; r < RPT; ++r) load_state<TPK, EXACT>(st + (long long)row(r) * N, lk, N, S[r]);
  }
  const float A = a.A[h], D = a.D != nullptr ? a.D[h] : 0.f, dtb = a.dt_bias != nullptr ? a.dt_bias[h] : 0.f;
  const long long go = (long long)(h / (a.H / a.G)) * N;
  for (long long t = t0; t < t0 + n; ++t) {
    const T *bp = a.Bm + t * a.ldb + go, *cp = a.Cm + t * a.ldc + go;
    float xv[RPT];
#pragma unroll
    for (int r = 0; r < RPT; ++r) xv[r] = ld1(a.x + t * a.ldx + (long long)h * a.P + row(r));
    float B[NPT], C[NPT];
    if constexpr (LIN) {                                   // the activations once per CTA
      __shared__ __align__(16) float sb[NP], sc[NP];
      if (t > t0) __syncthreads();
      for (int i = threadIdx.x; i < NP; i += 128) sb[i] = i < N ? silu_t<T>(ld1(bp + i)) : 0.f, sc[i] = i < N ? silu_t<T>(ld1(cp + i)) : 0.f;
      __syncthreads();
#pragma unroll
      for (int j = 0; j < NPT / 4; ++j) {
        const float4 b4 = *reinterpret_cast<const float4*>(&sb[4 * (lk + TPK * j)]), c4 = *reinterpret_cast<const float4*>(&sc[4 * (lk + TPK * j)]);
        B[4 * j] = b4.x, B[4 * j + 1] = b4.y, B[4 * j + 2] = b4.z, B[4 * j + 3] = b4.w;
        C[4 * j] = c4.x, C[4 * j + 1] = c4.y, C[4 * j + 2] = c4.z, C[4 * j + 3] = c4.w;
      }
    } else {
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
    }
    float d = A, dt = 1.f;
    if constexpr (!LIN) {
      dt = fminf(fmaxf(softplus_t<T>(ld1(a.dt + t * a.lddt + h) + dtb), a.dt_min), a.dt_max);
      d = exp_t<T>(dt * A);
    }
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const float u = LIN ? silu_t<T>(xv[r]) : dt * xv[r];
      float o[2] = {0.f, 0.f};
#pragma unroll
      for (int i = 0; i < NPT; ++i) {
        S[r][i] = fmaf(B[i], u, d * S[r][i]);
        o[i & 1] = fmaf(S[r][i], C[i], o[i & 1]);
      }
      const float tot = row_sum<TPK>(o[0] + o[1]);
      if (lk == 0 && p0 + RG * r < a.P) st1(a.y + t * a.ldy + (long long)h * a.P + p0 + RG * r, fmaf(D, xv[r], tot));
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
  // few sequences and heads: two rows per thread instead of four, so that twice as many SMs work
#define FLLM_SSD(T_, NP_, EXACT_, LIN_)                                                                                     \
  {                                                                                                                   \
    constexpr int drpt = LIN_ ? 2 : 1, drows = drpt * 128 / (NP_ / 16), rows4 = SsdTile<NP_, 4>::ROWS, rows2 = SsdTile<NP_, 2>::ROWS;             \
    const int tiles4 = p.H * ((p.P + rows4 - 1) / rows4), tiles2 = p.H * ((p.P + rows2 - 1) / rows2);                 \
    if (p.tokens == p.B)                                                                                              \
      launch_pdl(ssd_decode_kernel<T_, NP_, EXACT_, LIN_, drpt>, dim3(p.H * ((p.P + drows - 1) / drows), p.B), dim3(128), 0, stream, args(T_{}));  \
    else if (2LL * tiles4 * p.B <= sm_count() && tiles2 > tiles4)                                                     \
      launch_pdl(ssd_scan_kernel<T_, NP_, EXACT_, 2, LIN_>, dim3(tiles2, p.B), dim3(128), 0, stream, args(T_{}));           \
    else                                                                                                              \
      launch_pdl(ssd_scan_kernel<T_, NP_, EXACT_, 4, LIN_>, dim3(tiles4, p.B), dim3(128), 0, stream, args(T_{}));           \
    return 0;                                                                                                         \
  }
#define FLLM_SSD_N(T_, EXACT_, LIN_)                    \
  {                                                     \
    if (p.N <= 16) FLLM_SSD(T_, 16, EXACT_, LIN_)       \
    if (p.N <= 32) FLLM_SSD(T_, 32, EXACT_, LIN_)       \
    if (p.N <= 64) FLLM_SSD(T_, 64, EXACT_, LIN_)       \
    if (p.N <= 128) FLLM_SSD(T_, 128, EXACT_, LIN_)     \
    FLLM_SSD(T_, 256, EXACT_, LIN_)                     \
  }
  if (p.dt == nullptr) {               // constant decay
    if (p.f32) {
      if (exact) FLLM_SSD_N(float, true, true)
      FLLM_SSD_N(float, false, true)
    }
    if (exact) FLLM_SSD_N(bf16, true, true)
    FLLM_SSD_N(bf16, false, true)
  }
  if (p.f32) {
    if (exact) FLLM_SSD_N(float, true, false)
    FLLM_SSD_N(float, false, false)
  }
  if (exact) FLLM_SSD_N(bf16, true, false)
  FLLM_SSD_N(bf16, false, false)
#undef FLLM_SSD_N
#undef FLLM_SSD
}

}  // namespace fllm
