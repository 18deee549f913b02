// Recurrent token mixers on ragged batches: depthwise causal convolution, the Mamba-1 selective scan (Mamba-2: recurrent_ssd.cu)
// and the matrix-state family (RWKV-6, RWKV-7, gated delta rule, Kimi delta attention) plus the gated RMSNorm that
// follows a scan. The reference keeps one file per family (rust/engine/cuda/mamba1.cu, mamba2.cu, rwkv.cu,
// deltanet.cu, kda.cu, shortconv.cu) and a chunk-parallel scan (scan.cu); here every family walks its tokens with the
// state held in registers, one CTA per (sequence, head, slice of state rows): a step touches each state element
// once, so the work per token is the state size and the per-token inputs are prefetched a token or a chunk ahead. With 148 SMs
// the grid is sequences x heads x row tiles, which covers the machine from one 2048-token prefill chunk upwards.
//
// Batch layout (shared by every kernel): q_starts[B + 1] = first token row of each sequence, seq_state[B] = row of the
// state pool that belongs to the sequence, positions[T]: a sequence whose first token of the step sits at position 0
// starts from a zero state. States live in fp32 (convolution windows in bf16: they are copies of bf16 inputs).
#include <algorithm>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "fllm_ops.h"
#include "ptx.cuh"
#include "recurrent_util.cuh"
#include "tma_host.h"

namespace fllm {
namespace {
// ------------------------------------------------------------------------------------------ causal conv1d
// One CTA per (128 channels, sequence, run of `seg_tokens` tokens): the tokens of the run are spread over threadIdx.y,
// every thread owns two neighbouring channels. Only the CTA of a sequence's first run reads the sequence's window for
// its channels (later runs see their whole history in x, which nothing writes), so after a barrier that CTA moves the
// window forward in place. The last run of the grid goes on to the sequence's end.
template <typename T, int W>
__global__ void __launch_bounds__(256) conv1d_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ w,
                                                     const float* __restrict__ bias, T* __restrict__ state,
                                                     const int* __restrict__ q_starts, const int* __restrict__ seq_state,
                                                     const int* __restrict__ positions, T* __restrict__ y, long long ldy,
                                                     int C, int act, int seg_tokens) {
  pdl_wait();
  const int s = blockIdx.y;
  const int c = (blockIdx.x * 64 + threadIdx.x) * 2;
  const int t0 = q_starts[s], n = q_starts[s + 1] - t0;
  const int p_lo = blockIdx.z * seg_tokens, p_hi = blockIdx.z + 1 == gridDim.z ? n : min(n, p_lo + seg_tokens);
  if (n <= 0 || (p_lo >= n && blockIdx.z != 0)) return;
  const bool active = c < C;
  const bool fresh = positions[t0] == 0;
  T* st = state + (long long)seq_state[s] * (W - 1) * C;
  float wv[2][W], hist[2][W - 1], bv[2] = {0.f, 0.f};
  if (active) {
#pragma unroll
    for (int j = 0; j < W; ++j) wv[0][j] = w[(long long)c * W + j], wv[1][j] = w[(long long)(c + 1) * W + j];
    if (bias != nullptr) bv[0] = bias[c], bv[1] = bias[c + 1];
#pragma unroll
    for (int j = 0; j < W - 1; ++j) {
      float2 h = make_float2(0.f, 0.f);
      if (!fresh && blockIdx.z == 0) h = ld2(st + (long long)j * C + c);
      hist[0][j] = h.x, hist[1][j] = h.y;
    }
    // each row of threads walks a contiguous piece of the run with the last W - 1 inputs in registers: one load per token
    const int per = (p_hi - p_lo + (int)blockDim.y - 1) / (int)blockDim.y;
    const int a0 = p_lo + (int)threadIdx.y * per, a1 = min(p_hi, a0 + per);
    float win[2][W - 1];
#pragma unroll
    for (int j = 0; j < W - 1; ++j) {
      const int i = a0 - (W - 1) + j;
      float2 v = make_float2(0.f, 0.f);
      if (a0 < a1) {
        if (i >= 0) v = ld2(x + (long long)(t0 + i) * ldx + c);
        else v = make_float2(hist[0][(W - 1) + i], hist[1][(W - 1) + i]);
      }
      win[0][j] = v.x, win[1][j] = v.y;
    }
#pragma unroll 4
    for (int p = a0; p < a1; ++p) {
      const float2 v = ld2(x + (long long)(t0 + p) * ldx + c);
      float o0 = fmaf(wv[0][W - 1], v.x, bv[0]), o1 = fmaf(wv[1][W - 1], v.y, bv[1]);
#pragma unroll
      for (int j = 0; j < W - 1; ++j) o0 = fmaf(wv[0][j], win[0][j], o0), o1 = fmaf(wv[1][j], win[1][j], o1);
#pragma unroll
      for (int j = 0; j + 1 < W - 1; ++j) win[0][j] = win[0][j + 1], win[1][j] = win[1][j + 1];
      win[0][W - 2] = v.x, win[1][W - 2] = v.y;
      if (act) o0 = silu_t<T>(o0), o1 = silu_t<T>(o1);
      st2(y + (long long)(t0 + p) * ldy + c, o0, o1);
    }
  }
  if (blockIdx.z != 0) return;
  __syncthreads();
  if (active && threadIdx.y == 0) {
#pragma unroll
    for (int j = 0; j < W - 1; ++j) {
      const int i = n - (W - 1) + j;
      float2 v;
      if (i >= 0) v = ld2(x + (long long)(t0 + i) * ldx + c);
      else v = make_float2(hist[0][(W - 1) + i], hist[1][(W - 1) + i]);
      st2(st + (long long)j * C + c, v.x, v.y);
    }
  }
}

// Steps of single tokens (decode): one thread per two channels and sequence, every load in flight at once.
template <typename T, int W>
__global__ void __launch_bounds__(128) conv1d_decode_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ w,
                                                            const float* __restrict__ bias, T* __restrict__ state,
                                                            const int* __restrict__ q_starts, const int* __restrict__ seq_state,
                                                            const int* __restrict__ positions, T* __restrict__ y, long long ldy, int C, int act) {
  pdl_launch_dependents();
  const int s = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * 2;
  float wv[2][W], bv[2] = {0.f, 0.f};
  if (c < C) {                                               // weights do not wait for the kernel before
#pragma unroll
    for (int j = 0; j < W; ++j) wv[0][j] = w[(long long)c * W + j], wv[1][j] = w[(long long)(c + 1) * W + j];
    if (bias != nullptr) bv[0] = bias[c], bv[1] = bias[c + 1];
  }
  pdl_wait();
  const int t0 = q_starts[s], n = q_starts[s + 1] - t0;
  if (n <= 0 || c >= C) return;
  const bool fresh = positions[t0] == 0;
  T* st = state + (long long)seq_state[s] * (W - 1) * C + c;
  float2 win[W - 1];
#pragma unroll
  for (int j = 0; j < W - 1; ++j) win[j] = fresh ? make_float2(0.f, 0.f) : ld2(st + (long long)j * C);
  for (int p = 0; p < n; ++p) {
    const float2 v = ld2(x + (long long)(t0 + p) * ldx + c);
    float o0 = fmaf(wv[0][W - 1], v.x, bv[0]), o1 = fmaf(wv[1][W - 1], v.y, bv[1]);
#pragma unroll
    for (int j = 0; j < W - 1; ++j) o0 = fmaf(wv[0][j], win[j].x, o0), o1 = fmaf(wv[1][j], win[j].y, o1);
#pragma unroll
    for (int j = 0; j + 1 < W - 1; ++j) win[j] = win[j + 1];
    win[W - 2] = v;
    if (act) o0 = silu_t<T>(o0), o1 = silu_t<T>(o1);
    st2(y + (long long)(t0 + p) * ldy + c, o0, o1);
  }
#pragma unroll
  for (int j = 0; j < W - 1; ++j) st2(st + (long long)j * C, win[j].x, win[j].y);
}

// ------------------------------------------------------------------------------------------ Mamba-1
// h[d][n] = exp(dt[d] A[d][n]) h[d][n] + dt[d] B[n] x[d];  y[d] = (sum_n h[d][n] C[n] + D[d] x[d]) * silu(z[d])
//
// Long prompts of few sequences leave most SMs idle if a sequence is walked by one CTA per slice of channels. The recurrence
// is diagonal, so a sequence can be cut into segments of `seg_len` tokens that run side by side:
//   kLocal    every segment but the last runs from a zero state and leaves its end state and the sum of its time steps;
//   combine   start state of segment s + 1 = end state of s + exp(A sum dt_s) * start state of s (a short serial pass);
//   kFinal    every segment runs again from its true start state and writes y; the segment with the sequence's last token
//             stores the state. Sequences of one segment (decode rows of a mixed step) run only here, as the plain walk.
// Twice the arithmetic, `segs` times the parallelism. kWhole is the plain walk (decode, short chunks, large batches).
enum { kWhole = 0, kLocal = 1, kFinal = 2 };
struct Mamba1Args {
  const bf16 *x, *dt, *Bm, *Cm, *z;
  long long ldx, lddt, ldb, ldc, ldz, ldy;
  const float *A, *D, *dt_bias;   // A [Dm][N]
  float* state;                   // [slots][Dm][N]
  const int *q_starts, *seq_state, *positions;
  bf16* y;
  int Dm;
  int seg_len, segs;              // segmented modes only
  float* seg_state;               // [B][segs - 1][Dm][N]
  float* seg_start0;              // [B][Dm][N]: a continued sequence's state before the step (written by combine)
  float* seg_dt;                  // [B][segs - 1][Dm]: sum of a channel's time steps over a segment
};

template <int N, int MODE>
__global__ void __launch_bounds__(128) mamba1_scan_kernel(const Mamba1Args a) {
  const int d = blockIdx.x * 128 + threadIdx.x, s = blockIdx.y, seg = MODE == kWhole ? 0 : blockIdx.z;
  const int t0 = a.q_starts[s], n = a.q_starts[s + 1] - t0;
  if (n <= 0 || d >= a.Dm) return;
  float* st = a.state + ((long long)a.seq_state[s] * a.Dm + d) * N;
  const long long seg_stride = (long long)a.Dm * N;
  float* sg = MODE == kWhole ? nullptr : a.seg_state + ((long long)s * (a.segs - 1) * a.Dm + d) * N;
  const int seg_last = MODE == kWhole ? 0 : min(a.segs - 1, (n - 1) / a.seg_len);
  if ((MODE == kLocal && seg >= seg_last) || (MODE == kFinal && seg > seg_last)) return;
  const int lo = MODE == kWhole ? 0 : seg * a.seg_len;
  const int hi = (MODE == kWhole || (MODE == kFinal && seg == seg_last)) ? n : (seg + 1) * a.seg_len;
  float hs[N], A[N];
  load_f32<N>(a.A + (long long)d * N, A);
  const bool from_pool = MODE == kWhole || (MODE == kFinal && seg == 0);
  if (MODE == kLocal || (from_pool && a.positions[t0] == 0)) {
#pragma unroll
    for (int i = 0; i < N; ++i) hs[i] = 0.f;
  } else if (from_pool) {
    load_f32<N>(MODE == kFinal && seg_last > 0 ? a.seg_start0 + ((long long)s * a.Dm + d) * N : st, hs);
  } else {
    load_f32<N>(sg + (seg - 1) * seg_stride, hs);
  }
  const float D = a.D != nullptr ? a.D[d] : 0.f, dtb = a.dt_bias != nullptr ? a.dt_bias[d] : 0.f;
  float dt_sum = 0.f;
  for (int t = t0 + lo; t < t0 + hi; ++t) {
    float Bc[N], Cc[N];
    load_bf16<N>(a.Bm + (long long)t * a.ldb, Bc);           // the same words for the whole warp: one broadcast fetch
    if (MODE != kLocal) load_bf16<N>(a.Cm + (long long)t * a.ldc, Cc);
    const float xv = __bfloat162float(a.x[(long long)t * a.ldx + d]);
    const float dt = softplus_f(__bfloat162float(a.dt[(long long)t * a.lddt + d]) + dtb);
    const float dx = dt * xv;
    dt_sum += dt;
    if (MODE == kLocal) {
#pragma unroll
      for (int i = 0; i < N; ++i) hs[i] = fmaf(hs[i], __expf(dt * A[i]), dx * Bc[i]);
      continue;
    }
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      hs[i] = fmaf(hs[i], __expf(dt * A[i]), dx * Bc[i]);
      acc = fmaf(hs[i], Cc[i], acc);
    }
    acc = fmaf(D, xv, acc);
    if (a.z != nullptr) acc *= silu_f(__bfloat162float(a.z[(long long)t * a.ldz + d]));
    a.y[(long long)t * a.ldy + d] = __float2bfloat16(acc);
  }
  if (MODE == kLocal) {
    store_f32<N>(sg + seg * seg_stride, hs);
    a.seg_dt[((long long)s * (a.segs - 1) + seg) * a.Dm + d] = dt_sum;
  } else if (MODE == kWhole || seg == seg_last) {
    store_f32<N>(st, hs);
  }
}

// start[seg + 1] = end_local[seg] + exp(A sum dt[seg]) * start[seg] per channel and state entry, in place over seg_state
template <int N>
__global__ void mamba1_combine_kernel(const Mamba1Args a) {
  const int d = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y;
  const int t0 = a.q_starts[s];
  const int n = a.q_starts[s + 1] - t0;
  if (d >= a.Dm || n <= 0) return;
  const int seg_last = min(a.segs - 1, (n - 1) / a.seg_len);
  if (seg_last == 0) return;
  float carry[N], A[N];
  load_f32<N>(a.A + (long long)d * N, A);
  if (a.positions[t0] != 0) {
    load_f32<N>(a.state + ((long long)a.seq_state[s] * a.Dm + d) * N, carry);
    store_f32<N>(a.seg_start0 + ((long long)s * a.Dm + d) * N, carry);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) carry[i] = 0.f;
  }
  float* sg = a.seg_state + ((long long)s * (a.segs - 1) * a.Dm + d) * N;
  for (int seg = 0; seg < seg_last; ++seg) {
    const float sdt = a.seg_dt[((long long)s * (a.segs - 1) + seg) * a.Dm + d];
    float e[N];
    load_f32<N>(sg + (long long)seg * a.Dm * N, e);
#pragma unroll
    for (int i = 0; i < N; ++i) carry[i] = fmaf(carry[i], __expf(A[i] * sdt), e[i]);
    store_f32<N>(sg + (long long)seg * a.Dm * N, carry);
  }
}

// ------------------------------------------------------------------------------------------ matrix-state family
// State S[v][k] per head, one thread row per v with DK / NPT lanes along k. d = exp(w) is the decay.
//   kRwkv6      y = sum_k r (u k v + S);               S = S d + k v
//   kRwkv7      sa = sum_k S a;  S = S d + sa b + v k;   y = sum_k S r
//   kGatedDelta S = S d (one d per head);  m = sum_k S k;  S += k (v - m) beta;  y = sum_k S q
//   kKda        as kGatedDelta with one d per key channel
enum { kRwkv6 = 0, kRwkv7 = 1, kGatedDelta = 2, kKda = 3 };
template <typename T>
struct MatrixStateArgs {
  const T *r, *k, *v, *a, *b;     // r doubles as q; a, b only RWKV-7
  const float* w;                    // log decay: [T][H*DK] (per channel) or [T][H] (kGatedDelta)
  const float* u;                    // RWKV-6 bonus [H*DK]
  const T* beta;                  // [T][H] delta-rule step size (already through its sigmoid)
  long long ldr, ldk, ldv, lda, ldb, ldw, ldbeta, ldy;
  float* state;                      // [slots][H][DV][DK]
  const int *q_starts, *seq_state, *positions;
  T* y;
  int H, DV, kv_ratio;               // value heads per key head (q, k, w of head h come from head h / kv_ratio)
  int l2norm;                        // delta kinds: normalise q and k over DK inside the kernel
  float q_scale;
  // kGatedDelta with raw gates (w == nullptr): beta holds the logit of the step size, gate_raw [T][H] the logit a of the
  // decay; step size = sigmoid(beta), log decay = gate_A[h] * softplus(a + gate_dt_bias[h])
  const T* gate_raw;
  long long ldgate;
  const float *gate_A, *gate_dt_bias;
  int dk;                            // key width (delta_scan_kernel below a full one)
};

template <int KIND, int DK>
__global__ void __launch_bounds__(128) matrix_state_kernel(const MatrixStateArgs<bf16> a) {
  constexpr int NPT = 16, TPK = DK / NPT, ROWS = 128 / TPK;
  const int vtiles = (a.DV + ROWS - 1) / ROWS;
  const int h = blockIdx.x / vtiles, v = (blockIdx.x % vtiles) * ROWS + threadIdx.x / TPK;
  const int lk = threadIdx.x % TPK, s = blockIdx.y;
  const int t0 = a.q_starts[s], n = a.q_starts[s + 1] - t0;
  if (n <= 0) return;
  const bool valid = v < a.DV;
  const int vc = valid ? v : a.DV - 1;
  const int hk = h / a.kv_ratio;
  float* st = a.state + (((long long)a.seq_state[s] * a.H + h) * a.DV + vc) * DK + lk * NPT;
  float S[NPT];
  if (a.positions[t0] == 0) {
#pragma unroll
    for (int i = 0; i < NPT; ++i) S[i] = 0.f;
  } else {
    load_f32<NPT>(st, S);
  }
  float u[NPT];
  if (KIND == kRwkv6) load_f32<NPT>(a.u + (long long)hk * DK + lk * NPT, u);
  const long long ko = (long long)hk * DK + lk * NPT;
  for (int t = t0; t < t0 + n; ++t) {
    float r[NPT], k[NPT], d[NPT];
    load_bf16<NPT>(a.r + t * a.ldr + ko, r);
    load_bf16<NPT>(a.k + t * a.ldk + ko, k);
    const float vv = __bfloat162float(a.v[t * a.ldv + (long long)h * a.DV + vc]);
    load_f32<NPT>(a.w + t * a.ldw + ko, d);
#pragma unroll
    for (int i = 0; i < NPT; ++i) d[i] = __expf(d[i]);
    float out = 0.f;
    if (KIND == kRwkv6) {
#pragma unroll
      for (int i = 0; i < NPT; ++i) {
        const float kv = k[i] * vv;
        out = fmaf(r[i], fmaf(u[i], kv, S[i]), out);
        S[i] = fmaf(S[i], d[i], kv);
      }
      out = row_sum<TPK>(out);
    } else if (KIND == kRwkv7) {
      float av[NPT], bv[NPT], sa = 0.f;
      load_bf16<NPT>(a.a + t * a.lda + ko, av);
      load_bf16<NPT>(a.b + t * a.ldb + ko, bv);
#pragma unroll
      for (int i = 0; i < NPT; ++i) sa = fmaf(S[i], av[i], sa);
      sa = row_sum<TPK>(sa);
#pragma unroll
      for (int i = 0; i < NPT; ++i) {
        S[i] = fmaf(S[i], d[i], fmaf(sa, bv[i], vv * k[i]));
        out = fmaf(S[i], r[i], out);
      }
      out = row_sum<TPK>(out);
    } else {
      float qs = a.q_scale;
      if (a.l2norm) {
        float qq = 0.f, kk = 0.f;
#pragma unroll
        for (int i = 0; i < NPT; ++i) qq = fmaf(r[i], r[i], qq), kk = fmaf(k[i], k[i], kk);
        qq = row_sum<TPK>(qq), kk = row_sum<TPK>(kk);
        qs *= rsqrtf(qq + 1e-6f);
        const float ks = rsqrtf(kk + 1e-6f);
#pragma unroll
        for (int i = 0; i < NPT; ++i) k[i] *= ks;
      }
      float m = 0.f;
#pragma unroll
      for (int i = 0; i < NPT; ++i) {
        S[i] *= d[i];
        m = fmaf(S[i], k[i], m);
      }
      m = row_sum<TPK>(m);
      const float delta = (vv - m) * __bfloat162float(a.beta[t * a.ldbeta + h]);
#pragma unroll
      for (int i = 0; i < NPT; ++i) {
        S[i] = fmaf(k[i], delta, S[i]);
        out = fmaf(S[i], r[i], out);
      }
      out = row_sum<TPK>(out) * qs;
    }
    if (lk == 0 && valid) a.y[t * a.ldy + (long long)h * a.DV + vc] = __float2bfloat16(out);
  }
  if (valid) store_f32<NPT>(st, S);
}

// ------------------------------------------------------------------------------------------ gated delta rule
// One CTA per (sequence, head, ROWS value rows); TPK lanes share RPT rows, lane l holding the key columns 4 (l + TPK j) + 0..3
// of each (two rows per thread halve the shared-memory reads, which bound the walk).
// Tokens come in chunks of kDeltaChunk: eight threads per token fetch q and k one chunk ahead into registers, normalise them
// and leave them in shared memory as fp32 with the token's decay, step size and q . k, so the walk over a chunk touches
// shared memory only. With m = S k and o = S q of the state before the token (one pass, two sums side by side):
//   u = beta (v - d m);  S <- d S + u k;  y = d o + u (q . k)
// which is the read-out behind the token's write. DKP: key columns in registers; EXACT: the key width is DKP and rows are
// 16-byte aligned, otherwise it is a.dk <= DKP and rows are read value by value.
constexpr int kDeltaChunk = 16, kDeltaRows = 2;

template <typename T, int DKP, bool EXACT>
__global__ void __launch_bounds__(128) delta_scan_kernel(const MatrixStateArgs<T> a) {
  constexpr int NPT = 16, TPK = DKP / NPT, RPT = kDeltaRows, RG = 128 / TPK, ROWS = RPT * RG, C = kDeltaChunk, EPT = DKP / 8, VPT = ROWS * C / 128;
  __shared__ __align__(16) float sk[C][DKP], sq[C][DKP];
  __shared__ float sv[C][ROWS];
  __shared__ float4 sg[C];                               // decay, step size, q . k
  const int DK = EXACT ? DKP : a.dk;
  const int vtiles = (a.DV + ROWS - 1) / ROWS;
  const int h = blockIdx.x / vtiles, v0 = (blockIdx.x % vtiles) * ROWS, row = threadIdx.x / TPK;      // rows v0 + row + RG r
  const int lk = threadIdx.x % TPK, s = blockIdx.y;
  const int t0 = a.q_starts[s], n = a.q_starts[s + 1] - t0;
  if (n <= 0) return;
  float* st = a.state + ((long long)a.seq_state[s] * a.H + h) * a.DV * DK;
  float S[RPT][NPT];
  const bool fresh = a.positions[t0] == 0;
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
#pragma unroll
    for (int i = 0; i < NPT; ++i) S[r][i] = 0.f;
    if (!fresh) load_state<TPK, EXACT>(st + (long long)min(v0 + row + RG * r, a.DV - 1) * DK, lk, DK, S[r]);
  }
  // fetching: thread = (token tt of the chunk, share part of its row); values stay in their stored form until they are
  // staged, so that no conversion waits for the loads while the chunk before is walked. Shares are groups of eight values
  // (the shared-memory stores of a token's eight threads then spread over the banks).
  constexpr bool WIDE = EXACT && EPT % 8 == 0;
  constexpr int WORDS = WIDE ? EPT * (int)sizeof(T) / 16 : 1, LOOSE = WIDE ? 1 : EPT, PER8 = (int)sizeof(T) / 2;      // 16-byte words per group
  const int tt = threadIdx.x / 8, part = threadIdx.x % 8;
  const long long ko = (long long)(h / a.kv_ratio) * DK;
  auto column = [&](int i) { return EPT % 8 == 0 ? 8 * (part + 8 * (i / 8)) + i % 8 : part * EPT + i; };
  uint4 qw[WORDS], kw[WORDS];
  float ql[LOOSE], kl[LOOSE], wr = 0.f;
  T vr[VPT], gr{}, br{};
  auto fetch = [&](int base) {
    const int left = n - base;
    if (tt < left) {
      const long long t = t0 + base + tt;
      const T *qp = a.r + t * a.ldr + ko, *kp = a.k + t * a.ldk + ko;
      if constexpr (WIDE) {
#pragma unroll
        for (int i = 0; i < WORDS; ++i) {
          const int c = 8 * (part + 8 * (i / PER8)) + (i % PER8) * (16 / (int)sizeof(T));
          qw[i] = *reinterpret_cast<const uint4*>(qp + c);
          kw[i] = *reinterpret_cast<const uint4*>(kp + c);
        }
      } else {
#pragma unroll
        for (int i = 0; i < EPT; ++i) {
          const int c = column(i);
          ql[i] = c < DK ? ld1(qp + c) : 0.f;
          kl[i] = c < DK ? ld1(kp + c) : 0.f;
        }
      }
      if (part == 0) {
        if (a.w != nullptr) wr = a.w[t * a.ldw + h];
        else gr = a.gate_raw[t * a.ldgate + h];
        br = a.beta[t * a.ldbeta + h];
      }
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int e = threadIdx.x + i * 128, tv = e / ROWS, rv = min(v0 + e % ROWS, a.DV - 1);
      if (tv < left) vr[i] = a.v[(t0 + base + tv) * a.ldv + (long long)h * a.DV + rv];
    }
  };
  fetch(0);
  for (int base = 0; base < n; base += C) {
    const int cnt = min(C, n - base);
    __syncthreads();                                     // the chunk before is consumed
    {
      float qr[EPT], kr[EPT];
      if constexpr (WIDE) {
        const T *qt = reinterpret_cast<const T*>(qw), *kt = reinterpret_cast<const T*>(kw);
#pragma unroll
        for (int i = 0; i < EPT; ++i) qr[i] = ld1(qt + i), kr[i] = ld1(kt + i);
      } else {
#pragma unroll
        for (int i = 0; i < EPT; ++i) qr[i] = ql[i], kr[i] = kl[i];
      }
      float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int i = 0; i < EPT; ++i) qq = fmaf(qr[i], qr[i], qq), kk = fmaf(kr[i], kr[i], kk), qk = fmaf(qr[i], kr[i], qk);
      qq = row_sum<8>(qq), kk = row_sum<8>(kk), qk = row_sum<8>(qk);
      float qs = a.q_scale, ks = 1.f;
      if (a.l2norm) qs *= 1.f / sqrtf(qq + 1e-6f), ks = 1.f / sqrtf(kk + 1e-6f);
      if (tt < cnt) {
        if constexpr (EPT % 4 == 0) {
#pragma unroll
          for (int i = 0; i < EPT; i += 4) {
            *reinterpret_cast<float4*>(&sq[tt][column(i)]) = make_float4(qr[i] * qs, qr[i + 1] * qs, qr[i + 2] * qs, qr[i + 3] * qs);
            *reinterpret_cast<float4*>(&sk[tt][column(i)]) = make_float4(kr[i] * ks, kr[i + 1] * ks, kr[i + 2] * ks, kr[i + 3] * ks);
          }
        } else {
#pragma unroll
          for (int i = 0; i < EPT; ++i) sq[tt][column(i)] = qr[i] * qs, sk[tt][column(i)] = kr[i] * ks;
        }
        if (part == 0) {
          const bool raw = a.w == nullptr;
          sg[tt] = make_float4(exp_t<T>(raw ? a.gate_A[h] * softplus_t<T>(ld1(&gr) + a.gate_dt_bias[h]) : wr),
                               raw ? 1.f / (1.f + exp_t<T>(-ld1(&br))) : ld1(&br), qk * qs * ks, 0.f);
        }
      }
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int e = threadIdx.x + i * 128;
        if (e / ROWS < cnt) sv[e / ROWS][e % ROWS] = ld1(&vr[i]);
      }
    }
    __syncthreads();
    if (base + C < n) fetch(base + C);
    T* yp = a.y + (long long)(t0 + base) * a.ldy + (long long)h * a.DV + v0 + row;
    float4 kn[NPT / 4], qn[NPT / 4], gn = sg[0];           // the next token's rows travel while this one is applied
    float vn[RPT];
    auto rows_of = [&](int i) {
#pragma unroll
      for (int j = 0; j < NPT / 4; ++j) {
        kn[j] = *reinterpret_cast<const float4*>(&sk[i][4 * (lk + TPK * j)]);
        qn[j] = *reinterpret_cast<const float4*>(&sq[i][4 * (lk + TPK * j)]);
      }
      gn = sg[i];
#pragma unroll
      for (int r = 0; r < RPT; ++r) vn[r] = sv[i][row + RG * r];
    };
    rows_of(0);
#pragma unroll 2
    for (int i = 0; i < cnt; ++i, yp += a.ldy) {
      float4 k4[NPT / 4], q4[NPT / 4];
      float m2[RPT][2] = {}, o2[RPT][2] = {}, vv[RPT];
      const float d = gn.x, step = gn.y, kq = gn.z;
#pragma unroll
      for (int j = 0; j < NPT / 4; ++j) k4[j] = kn[j], q4[j] = qn[j];
#pragma unroll
      for (int r = 0; r < RPT; ++r) vv[r] = vn[r];
      rows_of(min(i + 1, cnt - 1));
#pragma unroll
      for (int j = 0; j < NPT / 4; ++j) {
        const float *kf = &k4[j].x, *qf = &q4[j].x;
#pragma unroll
        for (int r = 0; r < RPT; ++r)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            m2[r][e & 1] = fmaf(S[r][4 * j + e], kf[e], m2[r][e & 1]);
            o2[r][e & 1] = fmaf(S[r][4 * j + e], qf[e], o2[r][e & 1]);
          }
      }
#pragma unroll
      for (int r = 0; r < RPT; ++r) {
        const float m = row_sum<TPK>(m2[r][0] + m2[r][1]), o = row_sum<TPK>(o2[r][0] + o2[r][1]);
        const float u = step * fmaf(-d, m, vv[r]);
#pragma unroll
        for (int j = 0; j < NPT / 4; ++j) {
          const float* kf = &k4[j].x;
#pragma unroll
          for (int e = 0; e < 4; ++e) S[r][4 * j + e] = fmaf(kf[e], u, d * S[r][4 * j + e]);
        }
        if (lk == 0 && v0 + row + RG * r < a.DV) st1(yp + RG * r, fmaf(d, o, u * kq));
      }
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r)
    if (v0 + row + RG * r < a.DV) store_state<TPK, EXACT>(st + (long long)(v0 + row + RG * r) * DK, lk, DK, S[r]);
}

// The same recurrence for steps of single tokens (decode): one row per TPK lanes, inputs straight from global memory, no
// shared memory, so that many CTAs keep state reads in flight (a decoded token reads and writes the whole state once).
template <typename T, int DKP, bool EXACT>
__global__ void __launch_bounds__(128) delta_decode_kernel(const MatrixStateArgs<T> a) {
  constexpr int NPT = 16, TPK = DKP / NPT, ROWS = 128 / TPK;
  const int DK = EXACT ? DKP : a.dk;
  const int vtiles = (a.DV + ROWS - 1) / ROWS;
  const int h = blockIdx.x / vtiles, v = (blockIdx.x % vtiles) * ROWS + threadIdx.x / TPK;
  const int lk = threadIdx.x % TPK, s = blockIdx.y;
  const int t0 = a.q_starts[s], n = a.q_starts[s + 1] - t0;
  if (n <= 0) return;
  const int vc = min(v, a.DV - 1);
  float* st = a.state + (((long long)a.seq_state[s] * a.H + h) * a.DV + vc) * DK;
  float S[NPT];
#pragma unroll
  for (int i = 0; i < NPT; ++i) S[i] = 0.f;
  if (a.positions[t0] != 0) load_state<TPK, EXACT>(st, lk, DK, S);
  const bool raw = a.w == nullptr;
  for (long long t = t0; t < t0 + n; ++t) {
    const T *qp = a.r + t * a.ldr + (long long)(h / a.kv_ratio) * DK, *kp = a.k + t * a.ldk + (long long)(h / a.kv_ratio) * DK;
    float q[NPT], k[NPT];
#pragma unroll
    for (int j = 0; j < NPT / 4; ++j) {
      const int c = 4 * (lk + TPK * j);
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        float2 q2 = make_float2(0.f, 0.f), k2 = q2;
        if (EXACT) {
          q2 = ld2(qp + c + e), k2 = ld2(kp + c + e);
        } else {
          if (c + e < DK) q2.x = ld1(qp + c + e), k2.x = ld1(kp + c + e);
          if (c + e + 1 < DK) q2.y = ld1(qp + c + e + 1), k2.y = ld1(kp + c + e + 1);
        }
        q[4 * j + e] = q2.x, q[4 * j + e + 1] = q2.y, k[4 * j + e] = k2.x, k[4 * j + e + 1] = k2.y;
      }
    }
    const float g = raw ? ld1(a.gate_raw + t * a.ldgate + h) : a.w[t * a.ldw + h], b = ld1(a.beta + t * a.ldbeta + h);
    const float vv = ld1(a.v + t * a.ldv + (long long)h * a.DV + vc);
    float qq = 0.f, kk = 0.f, qk = 0.f, m = 0.f, o = 0.f;
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
      qq = fmaf(q[i], q[i], qq), kk = fmaf(k[i], k[i], kk), qk = fmaf(q[i], k[i], qk);
      m = fmaf(S[i], k[i], m), o = fmaf(S[i], q[i], o);
    }
    qk = row_sum<TPK>(qk), m = row_sum<TPK>(m), o = row_sum<TPK>(o);
    float qs = a.q_scale, ks = 1.f;
    if (a.l2norm) qs *= 1.f / sqrtf(row_sum<TPK>(qq) + 1e-6f), ks = 1.f / sqrtf(row_sum<TPK>(kk) + 1e-6f);
    const float d = exp_t<T>(raw ? a.gate_A[h] * softplus_t<T>(g + a.gate_dt_bias[h]) : g), step = raw ? 1.f / (1.f + exp_t<T>(-b)) : b;
    const float u = step * fmaf(-d, m * ks, vv);
#pragma unroll
    for (int i = 0; i < NPT; ++i) S[i] = fmaf(k[i] * ks, u, d * S[i]);
    if (lk == 0 && v < a.DV) st1(a.y + t * a.ldy + (long long)h * a.DV + v, qs * fmaf(d, o, u * qk * ks));
  }
  if (v < a.DV) store_state<TPK, EXACT>(st, lk, DK, S);
}

// ------------------------------------------------------------------------------------------ gated RMSNorm
// Per (token, group of `gs` channels): mode 0  y = rmsnorm(x * silu(z)) * w   (Mamba-2: gate first)
//                                      mode 1  y = rmsnorm(x) * w * silu(z)   (gated delta net: norm first)
// w has `wlen` entries (D for Mamba-2, the head width when every head shares one weight). One warp per group.
// y may be x (every element is read and then written by the same thread).
// mode: bit 0 = the norm comes before the gate, bit 1 = the gate is sigmoid(z) instead of silu(z)
template <typename T>
__device__ __forceinline__ float gate_t(float z, int mode) {
  return ((mode & 2) ? 1.f : z) / (1.f + exp_t<T>(-z));
}
template <typename T>
__global__ void __launch_bounds__(128) gated_rmsnorm_kernel(const T* x, long long ldx, const T* __restrict__ z, long long ldz,
                                                            const T* __restrict__ w, int wlen, T* y, long long ldy, int n_rows, int D,
                                                            int gs, float eps, int mode) {
  pdl_launch_dependents();
  pdl_wait();
  const int groups = D / gs;
  const long long item = (long long)blockIdx.x * 4 + threadIdx.x / 32;
  if (item >= (long long)n_rows * groups) return;
  const int t = (int)(item / groups), g = (int)(item % groups), lane = threadIdx.x % 32;
  const T* xr = x + t * ldx + (long long)g * gs;
  const T* zr = z != nullptr ? z + t * ldz + (long long)g * gs : nullptr;
  float ss = 0.f;
  for (int i = lane; i < gs; i += 32) {
    float v = ld1(xr + i);
    if ((mode & 1) == 0 && zr != nullptr) v *= gate_t<T>(ld1(zr + i), mode);
    ss = fmaf(v, v, ss);
  }
  ss = row_sum<32>(ss);
  const float inv = sizeof(T) == 4 ? 1.f / sqrtf(ss / gs + eps) : rsqrtf(ss / gs + eps);
  T* yr = y + t * ldy + (long long)g * gs;
  for (int i = lane; i < gs; i += 32) {
    float v = ld1(xr + i);
    const float gate = zr != nullptr ? gate_t<T>(ld1(zr + i), mode) : 1.f;
    if ((mode & 1) == 0) v *= gate;
    v = v * inv * ld1(w + (g * gs + i) % wlen);
    if ((mode & 1)) v *= gate;
    st1(yr + i, v);
  }
}

// The same for wide groups (Mamba-2 normalises up to the whole inner width at once): one CTA per (token, group), two channels
// per thread and step, the (gated) row kept in registers between the two passes when it fits (2 * THREADS * KEEP channels).
template <int THREADS, int KEEP>
__global__ void __launch_bounds__(THREADS) gated_rmsnorm_wide_kernel(const bf16* x, long long ldx, const bf16* __restrict__ z, long long ldz,
                                                                     const bf16* __restrict__ w, int wlen, bf16* y, long long ldy, int D, int gs,
                                                                     float eps, int mode) {
  pdl_launch_dependents();
  pdl_wait();
  const int groups = D / gs;
  const int t = blockIdx.x / groups, g = blockIdx.x % groups;
  const __nv_bfloat162* xr = reinterpret_cast<const __nv_bfloat162*>(x + t * ldx + (long long)g * gs);
  const __nv_bfloat162* zr = z != nullptr ? reinterpret_cast<const __nv_bfloat162*>(z + t * ldz + (long long)g * gs) : nullptr;
  const int pairs = gs / 2;
  float2 keep[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int p = threadIdx.x + i * THREADS;
    keep[i] = make_float2(0.f, 0.f);
    if (p < pairs) {
      keep[i] = __bfloat1622float2(xr[p]);
      if ((mode & 1) == 0 && zr != nullptr) {
        const float2 zz = __bfloat1622float2(zr[p]);
        keep[i].x *= gate_t<bf16>(zz.x, mode), keep[i].y *= gate_t<bf16>(zz.y, mode);
      }
      ss = fmaf(keep[i].x, keep[i].x, fmaf(keep[i].y, keep[i].y, ss));
    }
  }
  for (int p = threadIdx.x + KEEP * THREADS; p < pairs; p += THREADS) {     // beyond the kept part: read again in the second pass
    float2 v = __bfloat1622float2(xr[p]);
    if ((mode & 1) == 0 && zr != nullptr) {
      const float2 zz = __bfloat1622float2(zr[p]);
      v.x *= gate_t<bf16>(zz.x, mode), v.y *= gate_t<bf16>(zz.y, mode);
    }
    ss = fmaf(v.x, v.x, fmaf(v.y, v.y, ss));
  }
  __shared__ float part[THREADS / 32];
  ss = row_sum<32>(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) tot += part[i];
  const float inv = rsqrtf(tot / gs + eps);
  __nv_bfloat162* yr = reinterpret_cast<__nv_bfloat162*>(y + t * ldy + (long long)g * gs);
  const int w0 = (g * gs) % wlen;
  auto weight = [&](int p) {
    int c = w0 + 2 * p, d = c + 1;
    if (d >= wlen) c %= wlen, d %= wlen;
    return make_float2(__bfloat162float(w[c]), __bfloat162float(w[d]));
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int p = threadIdx.x + i * THREADS;
    if (p < pairs) {
      const float2 ww = weight(p);
      float2 v = make_float2(keep[i].x * inv * ww.x, keep[i].y * inv * ww.y);
      if ((mode & 1) && zr != nullptr) {
        const float2 zz = __bfloat1622float2(zr[p]);
        v.x *= gate_t<bf16>(zz.x, mode), v.y *= gate_t<bf16>(zz.y, mode);
      }
      yr[p] = __floats2bfloat162_rn(v.x, v.y);
    }
  }
  for (int p = threadIdx.x + KEEP * THREADS; p < pairs; p += THREADS) {
    float2 v = __bfloat1622float2(xr[p]);
    float2 gt = make_float2(1.f, 1.f);
    if (zr != nullptr) {
      const float2 zz = __bfloat1622float2(zr[p]);
      gt = make_float2(gate_t<bf16>(zz.x, mode), gate_t<bf16>(zz.y, mode));
    }
    if ((mode & 1) == 0) v.x *= gt.x, v.y *= gt.y;
    const float2 ww = weight(p);
    v = make_float2(v.x * inv * ww.x, v.y * inv * ww.y);
    if ((mode & 1)) v.x *= gt.x, v.y *= gt.y;
    yr[p] = __floats2bfloat162_rn(v.x, v.y);
  }
}

}  // namespace

// ---------------------------------------------------------------------------------------------- launchers
// Every launcher returns 0 on success or a negative code naming the argument it rejected, before any launch.
int causal_conv1d(const void* x, long long ldx, const float* w, const float* bias, void* state, const int* q_starts,
                  const int* seq_state, const int* positions, void* y, long long ldy, int B, int C, int W, int act,
                  int tokens, int max_q_len, cudaStream_t stream, int f32) {
  if (B <= 0) return 0;
  if (C % 2 || (ldx % 2) || (ldy % 2) || x == y) return -1;
  if (W < 2 || W > 8) return -2;
  constexpr int seg_tokens = 64;                       // 16 tokens per thread
  const int runs = std::min(std::max((max_q_len + seg_tokens - 1) / seg_tokens, 1), 65535);
  const dim3 grid((C / 2 + 63) / 64, B, runs), block(64, 4);
  auto go = [&](auto zero) {
    using T = decltype(zero);
    auto xs = static_cast<const T*>(x);
    auto ys = static_cast<T*>(y);
    auto ss = static_cast<T*>(state);
#define FLLM_CONV(W_)                                                                                                                               \
  case W_:                                                                                                                                          \
    if (tokens == B)                                                                                                                                \
      launch_pdl(conv1d_decode_kernel<T, W_>, dim3((C / 2 + 127) / 128, B), dim3(128), 0, stream, xs, ldx, w, bias, ss, q_starts, seq_state, positions, ys, \
                 ldy, C, act);                                                                                                                      \
    else                                                                                                                                            \
      launch_pdl(conv1d_kernel<T, W_>, grid, block, 0, stream, xs, ldx, w, bias, ss, q_starts, seq_state, positions, ys, ldy, C, act, (int)seg_tokens);   \
    break;
    switch (W) { FLLM_CONV(2) FLLM_CONV(3) FLLM_CONV(4) FLLM_CONV(5) FLLM_CONV(6) FLLM_CONV(7) FLLM_CONV(8) }
#undef FLLM_CONV
  };
  if (f32) go(float{});
  else go(bf16{});
  return 0;
}

// seg_len > 0 with segs > 1: the sequence-parallel form (seg_state: B * segs * Dm * N floats, seg_dt: B * (segs - 1) * Dm floats);
// segs must cover the longest sequence of the step (segs * seg_len >= its tokens).
int mamba1_scan(const void* x, long long ldx, const void* dt, long long lddt, const void* Bm, long long ldb, const void* Cm,
                long long ldc, const void* z, long long ldz, const float* A, const float* D, const float* dt_bias, float* state,
                const int* q_starts, const int* seq_state, const int* positions, void* y, long long ldy, int B, int Dm, int N,
                int seg_len, int segs, float* seg_state, float* seg_dt, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (!aligned16(Bm) || !aligned16(Cm) || (ldb % 8) || (ldc % 8)) return -1;
  const bool segmented = seg_len > 0 && segs > 1;
  if (segmented && (seg_state == nullptr || seg_dt == nullptr || !aligned16(seg_state))) return -3;
  Mamba1Args a{static_cast<const bf16*>(x), static_cast<const bf16*>(dt), static_cast<const bf16*>(Bm), static_cast<const bf16*>(Cm),
               static_cast<const bf16*>(z), ldx, lddt, ldb, ldc, ldz, ldy, A, D, dt_bias, state, q_starts, seq_state, positions,
               static_cast<bf16*>(y), Dm, seg_len, segs, seg_state,
               segmented ? seg_state + (long long)B * (segs - 1) * Dm * N : nullptr, seg_dt};
  const unsigned gx = (Dm + 127) / 128;
#define FLLM_M1(N_)                                                                           \
  {                                                                                           \
    if (!segmented) {                                                                         \
      mamba1_scan_kernel<N_, kWhole><<<dim3(gx, B), 128, 0, stream>>>(a);                     \
    } else {                                                                                  \
      mamba1_scan_kernel<N_, kLocal><<<dim3(gx, B, segs - 1), 128, 0, stream>>>(a);           \
      mamba1_combine_kernel<N_><<<dim3(gx, B), 128, 0, stream>>>(a);                          \
      mamba1_scan_kernel<N_, kFinal><<<dim3(gx, B, segs), 128, 0, stream>>>(a);               \
    }                                                                                         \
    return 0;                                                                                 \
  }
  if (N == 16) FLLM_M1(16)
  if (N == 8) FLLM_M1(8)
#undef FLLM_M1
  return -2;
}

int matrix_state_scan(int kind, const void* r, long long ldr, const void* k, long long ldk, const void* v, long long ldv,
                      const void* a_, long long lda, const void* b_, long long ldb, const float* w, long long ldw, const float* u,
                      const void* beta, long long ldbeta, float* state, const int* q_starts, const int* seq_state,
                      const int* positions, void* y, long long ldy, int B, int H, int DK, int DV, int kv_ratio, int l2norm,
                      float q_scale, const void* gate_raw, long long ldgate, const float* gate_A, const float* gate_dt_bias,
                      int tokens, cudaStream_t stream, int f32) {
  if (B <= 0) return 0;
  if (kv_ratio <= 0 || H % kv_ratio || DK <= 0) return -1;
  const int unit = f32 ? 4 : 8;
  const bool exact = (DK == 16 || DK == 32 || DK == 64 || DK == 128 || DK == 256) && aligned16(r) && aligned16(k) && ldr % unit == 0 && ldk % unit == 0;
  if (w == nullptr && (kind != kGatedDelta || gate_raw == nullptr || gate_A == nullptr || gate_dt_bias == nullptr)) return -4;
  if (kind != kGatedDelta && (!exact || DK == 16 || f32)) return exact ? -2 : -1;       // the other kinds: bf16, full key widths
  if (kind != kGatedDelta && (!aligned16(w) || (ldw % 4))) return -1;
  if (kind == kRwkv7 && (!aligned16(a_) || !aligned16(b_) || (lda % 8) || (ldb % 8))) return -1;
  if (kind == kRwkv6 && !aligned16(u)) return -1;
  if (DK > 256) return -2;
  auto args = [&](auto zero) {
    using T = decltype(zero);
    return MatrixStateArgs<T>{static_cast<const T*>(r), static_cast<const T*>(k), static_cast<const T*>(v), static_cast<const T*>(a_),
                              static_cast<const T*>(b_), w, u, static_cast<const T*>(beta), ldr, ldk, ldv, lda, ldb, ldw, ldbeta, ldy, state,
                              q_starts, seq_state, positions, static_cast<T*>(y), H, DV, kv_ratio, l2norm, q_scale,
                              static_cast<const T*>(gate_raw), ldgate, gate_A, gate_dt_bias, DK};
  };
#define FLLM_MS(KIND_, DK_)                                                                                          \
  {                                                                                                                  \
    constexpr int rows = 128 / (DK_ / 16);                                                                           \
    matrix_state_kernel<KIND_, DK_><<<dim3(H * ((DV + rows - 1) / rows), B), 128, 0, stream>>>(args(bf16{}));        \
    return 0;                                                                                                        \
  }
#define FLLM_MS_DK(KIND_)           \
  switch (DK) {                     \
    case 32: FLLM_MS(KIND_, 32)     \
    case 64: FLLM_MS(KIND_, 64)     \
    case 128: FLLM_MS(KIND_, 128)   \
    case 256: FLLM_MS(KIND_, 256)   \
    default: return -2;             \
  }
#define FLLM_DS(T_, DK_, EXACT_)                                                                                     \
  {                                                                                                                  \
    constexpr int rows = 128 / (DK_ / 16);                                                                           \
    if (tokens == B)                                                                                                 \
      delta_decode_kernel<T_, DK_, EXACT_><<<dim3(H * ((DV + rows - 1) / rows), B), 128, 0, stream>>>(args(T_{}));   \
    else                                                                                                             \
      delta_scan_kernel<T_, DK_, EXACT_><<<dim3(H * ((DV + kDeltaRows * rows - 1) / (kDeltaRows * rows)), B), 128, 0, stream>>>(args(T_{})); \
    return 0;                                                                                                        \
  }
#define FLLM_GD(T_, EXACT_)                  \
  {                                          \
    if (DK <= 16) FLLM_DS(T_, 16, EXACT_)    \
    if (DK <= 32) FLLM_DS(T_, 32, EXACT_)    \
    if (DK <= 64) FLLM_DS(T_, 64, EXACT_)    \
    if (DK <= 128) FLLM_DS(T_, 128, EXACT_)  \
    FLLM_DS(T_, 256, EXACT_)                 \
  }
  switch (kind) {
    case kRwkv6: FLLM_MS_DK(kRwkv6)
    case kRwkv7: FLLM_MS_DK(kRwkv7)
    case kKda: FLLM_MS_DK(kKda)
    case kGatedDelta:
      if (f32) {
        if (exact) FLLM_GD(float, true)
        FLLM_GD(float, false)
      }
      if (exact) FLLM_GD(bf16, true)
      FLLM_GD(bf16, false)
  }
#undef FLLM_GD
#undef FLLM_DS
#undef FLLM_MS_DK
#undef FLLM_MS
  return -3;
}

void gated_rmsnorm(const void* x, long long ldx, const void* z, long long ldz, const void* w, int wlen, void* y, long long ldy, int T,
                   int D, int group_size, float eps, int norm_before_gate, cudaStream_t stream, int f32, int sigmoid_gate) {
  if (T <= 0) return;
  const int mode = norm_before_gate | (sigmoid_gate << 1);
  const long long items = (long long)T * (D / group_size);
  if (f32) {
    gated_rmsnorm_kernel<float><<<(unsigned)((items + 3) / 4), 128, 0, stream>>>(
        static_cast<const float*>(x), ldx, static_cast<const float*>(z), ldz, static_cast<const float*>(w), wlen, static_cast<float*>(y), ldy, T, D,
        group_size, eps, mode);
    return;
  }
  const bool pairs_ok = group_size % 2 == 0 && ldx % 2 == 0 && ldy % 2 == 0 && (z == nullptr || ldz % 2 == 0) &&
                        (reinterpret_cast<uintptr_t>(x) & 3) == 0 && (reinterpret_cast<uintptr_t>(y) & 3) == 0 &&
                        (reinterpret_cast<uintptr_t>(z) & 3) == 0;
  auto go = [&](auto kernel, unsigned grid, unsigned threads) {
    launch_pdl(kernel, dim3(grid), dim3(threads), 0, stream, static_cast<const bf16*>(x), ldx, static_cast<const bf16*>(z), ldz, static_cast<const bf16*>(w), wlen,
               static_cast<bf16*>(y), ldy, D, group_size, eps, mode);
  };
  if (group_size > 4096 && pairs_ok) go(gated_rmsnorm_wide_kernel<256, 16>, (unsigned)items, 256);
  else if (group_size > 2048 && pairs_ok) go(gated_rmsnorm_wide_kernel<256, 8>, (unsigned)items, 256);
  else if (group_size > 1024 && pairs_ok) go(gated_rmsnorm_wide_kernel<256, 4>, (unsigned)items, 256);
  else if (group_size > 256 && pairs_ok) go(gated_rmsnorm_wide_kernel<128, 4>, (unsigned)items, 128);
  else
    launch_pdl(gated_rmsnorm_kernel<bf16>, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, stream, static_cast<const bf16*>(x), ldx, static_cast<const bf16*>(z), ldz,
               static_cast<const bf16*>(w), wlen, static_cast<bf16*>(y), ldy, T, D, group_size, eps, mode);
}

}  // namespace fllm
