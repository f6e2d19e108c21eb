// Recurrent mixers of the ragged serving step: short causal convolutions with a carried tail, and linear-attention state
// scans (a decayed outer-product state, and the gated delta rule), all in fp32.
//
// A step is a flat list of tokens; token t sits at position pos[t] of the sequence in state row slot[t]. The tokens of one
// sequence are consecutive and form a run; `runs` int32 [n_runs, 4] = (first row, rows, position of the first row, state
// row), or NULL: every token is a run of its own (a decode batch, read from pos / slot on the device). A run that starts
// at position 0 starts from a zero state whatever its state row held before, so rows are reused without clearing.
//
//   b200_short_conv        y[t, c] = act(sum_j w[c, j] x[t - (taps - 1) + j, c]); inputs before the run come from the tail
//                          kept in `state` [rows, taps - 1, C] (the last taps - 1 inputs; zeros before position 0).
//   b200_silu_rows         x <- silu(x) in place on a column slice of fp32 rows (the activation of projections that enter a
//                          scan without a convolution, done once instead of by every CTA that reads them).
//   b200_short_conv_tail   advances that tail over the step's runs (launched after the convolution has read the old one); for
//                          a decode batch the convolution does it itself. `in_bias`: a bias that belongs to the inputs.
//   b200_delta_gates       q, k -> unit vectors per head (q also times `qscale`); a -> exp(-exp(A_log[h]) softplus(a + bias)),
//                          one per key channel or one per head; b -> sigmoid(b); in place, fp32.
//   b200_token_shift       several mixes of every token with the one before it, h + (h' - h) mu_s, h' carried like a tail.
//   b200_linear_scan       per head, state S [D, Dv] (fp32, in `state` [rows, H, D, Dv]):
//                            mode 0  S <- decay_h S + k v^T ;                                   o = S^T q
//                            mode 1  S <- diag(g) S ; u = beta (v - S^T k) ; S <- S + k u^T ;   o = S^T q
//                            mode 2  S <- a_t S + b_t k v^T  (a, b one number per token and head) ;   o = S^T q
//                            mode 3  mode 1 with one decay per token and head
//                          `ones` appends a column of ones to v (the state's last column is then the decayed sum of the
//                          b_t k_t, and o's last column its product with q: the normaliser of an mLSTM read-out).
//   b200_mlstm_gates       capped log gates of an mLSTM with their running maximum m (carried per sequence and head):
//                          i = cap tanh((gi + bi) / cap), f = logsigmoid(cap tanh((gf + bf) / cap)), m' = max(f + m, i);
//                          a = exp(f + m - m'), b = exp(i - m'), e = exp(-m'). m = 0 before position 0.
//   b200_ssm_gates         step sizes of a selective state space: dt = softplus(x + bias), a = exp(-exp(A_log) dt), b = dt.
//   b200_scan_readout      what follows a scan per token: optional division of each head by max(|last column|, e) + den_eps,
//                          optional skip D_h x, optional silu gate BEFORE the norm, RMS norm over equal column groups,
//                          weight (one per column, or shared by the groups), optional sigmoid or silu gate AFTER the norm.
//                          Columns of S are independent, so a thread owns R rows of one column, the lanes that share a
//                          column reduce their partial dot products by shuffles, and a CTA owns a block of columns of one
//                          (run, head): tokens are walked in order, staged through shared memory in chunks.
#include "common.cuh"
#include "../include/b200_ops.h"

namespace b200 {

__device__ __forceinline__ float silu_f(float v) { return v / (1.f + expf(-v)); }

// V = 1 or 4 neighbouring elements as fp32 (V = 4: on a boundary of four elements)
template <int V, typename T> __device__ __forceinline__ void load_f32(const T* p, float (&v)[V]) {
  if (V == 4 && sizeof(T) == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
  else if (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(raw.x), b = unpack_bf16x2(raw.y);
    v[0] = a.x; v[V > 1 ? 1 : 0] = a.y; v[V > 2 ? 2 : 0] = b.x; v[V - 1] = b.y;
  } else v[0] = to_f32<T>(p[0]);
}

// V channels per thread (V = 4: rows of x, y, the tail and C are multiples of four floats on 16-byte boundaries)
// step_tail: every token is a run of its own, so the thread that reads a channel's old tail also advances it
template <int V, typename TX, typename TY>
__global__ void short_conv_kernel(const TX* __restrict__ x, long long ldx, const float* __restrict__ w,
                                  const float* __restrict__ bias, float* __restrict__ state, const int* __restrict__ pos,
                                  const int* __restrict__ slot, TY* __restrict__ y, long long ldy, int tokens, int C, int taps,
                                  int act, int residual, int step_tail) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int CV = C / V;
  if (idx >= (long long)tokens * CV) return;
  const int t = (int)(idx / CV), c = (int)(idx % CV) * V;
  const int p = pos[t], s = slot[t];
  // nb: tokens of the same run right before t (at most taps - 1 matter)
  int nb = 0;
  if (!step_tail)
    while (nb < taps - 1 && t - nb - 1 >= 0 && slot[t - nb - 1] == s) ++nb;
  float acc[V], own[V], prev[V];
#pragma unroll
  for (int e = 0; e < V; ++e) { acc[e] = bias ? bias[c + e] : 0.f; own[e] = 0.f; prev[e] = 0.f; }
  for (int d = 0; d < taps; ++d) {                       // d tokens back
    if (p - d < 0 && !step_tail) break;
    float v[V];
    float* old = state + ((long long)s * (taps - 1) + (taps - 1 - (d - nb))) * C + c;      // read where d > nb
    if (p - d < 0) {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = 0.f;
    } else if (d <= nb) {
      load_f32<V, TX>(x + (long long)(t - d) * ldx + c, v);
    } else {
      load_f32<V, float>(old, v);
    }
    if (step_tail && d > 0) {                            // entry taps - 1 - d held the input d tokens back: it takes the next one
#pragma unroll
      for (int e = 0; e < V; ++e) old[e] = prev[e];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      acc[e] = fmaf(w[(long long)(c + e) * taps + (taps - 1 - d)], v[e], acc[e]);
      if (d == 0) own[e] = v[e];
      prev[e] = v[e];
    }
  }
#pragma unroll
  for (int e = 0; e < V; ++e) acc[e] = (act ? silu_f(acc[e]) : acc[e]) + (residual ? own[e] : 0.f);
  TY* dst = y + (long long)t * ldy + c;
  if (V == 4 && sizeof(TY) == 4) *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(acc);
  else if (V == 4) *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(acc[0], acc[1 % V]), pack_bf16x2(acc[V - 2 >= 0 ? V - 2 : 0], acc[V - 1]));
  else {
#pragma unroll
    for (int e = 0; e < V; ++e) dst[e] = from_f32<TY>(acc[e]);
  }
}

// The same over prompt pieces, for few taps: a thread owns V channels over TB consecutive tokens, keeps their weights and last
// TAPS - 1 inputs in registers, and fetches what lies before a token only where a run starts (from x, the tail, or zeros).
template <int V, typename TX, typename TY, int TAPS>
__global__ void __launch_bounds__(128)
short_conv_run_kernel(const TX* __restrict__ x, long long ldx, const float* __restrict__ w, const float* __restrict__ bias,
                      const float* __restrict__ state, const int* __restrict__ pos, const int* __restrict__ slot, TY* __restrict__ y,
                      long long ldy, int tokens, int C, int act, int residual, int TB) {
  constexpr int L = TAPS - 1, LH = L > 0 ? L : 1;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  float wt[TAPS][V], hist[LH][V], b[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    b[e] = bias ? bias[c + e] : 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wt[j][e] = w[(long long)(c + e) * TAPS + j];
#pragma unroll
    for (int j = 0; j < LH; ++j) hist[j][e] = 0.f;
  }
  const int t0 = blockIdx.y * TB, t1 = min(tokens, t0 + TB);
  int ps = -1, pp = -2;
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    const int p = pos[t], s = slot[t];
    if (L > 0 && !(s == ps && p == pp + 1)) {
      int nb = 0;
      while (nb < L && t - nb - 1 >= 0 && slot[t - nb - 1] == s && pos[t - nb - 1] == p - nb - 1) ++nb;
#pragma unroll
      for (int d = 1; d <= L; ++d) {                       // d tokens back -> hist[L - d]
        float v[V];
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = 0.f;
        if (p - d >= 0) {
          if (d <= nb) load_f32<V, TX>(x + (long long)(t - d) * ldx + c, v);
          else load_f32<V, float>(state + ((long long)s * L + (L - (d - nb))) * C + c, v);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) hist[L > 0 ? L - d : 0][e] = v[e];
      }
    }
    ps = s; pp = p;
    float v[V], a[V];
    load_f32<V, TX>(x + (long long)t * ldx + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      float acc = b[e];
#pragma unroll
      for (int j = 0; j < L; ++j) acc = fmaf(wt[j][e], hist[j][e], acc);
      acc = fmaf(wt[TAPS - 1][e], v[e], acc);
#pragma unroll
      for (int j = 0; j + 1 < L; ++j) hist[j][e] = hist[j + 1][e];
      if (L > 0) hist[LH - 1][e] = v[e];
      if (act) acc = sizeof(TY) == 4 ? silu_f(acc) : __fdividef(acc, 1.f + __expf(-acc));
      a[e] = acc + (residual ? v[e] : 0.f);
    }
    TY* dst = y + (long long)t * ldy + c;
    if (V == 4 && sizeof(TY) == 4) *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(a);
    else if (V == 4) *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(a[0], a[1 % V]), pack_bf16x2(a[V - 2 >= 0 ? V - 2 : 0], a[V - 1]));
    else dst[0] = from_f32<TY>(a[0]);
  }
}

constexpr int kMaxTaps = 16;

// x[r, c] <- silu(x[r, c]) over the first `cols` columns of rows of stride ld
template <int V>
__global__ void silu_rows_kernel(float* __restrict__ x, long long ld, long long rows, int cols) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int CV = cols / V;
  if (idx >= rows * CV) return;
  float* px = x + (idx / CV) * ld + (idx % CV) * V;
  float v[V];
  if (V == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(px);
  else v[0] = px[0];
#pragma unroll
  for (int e = 0; e < V; ++e) v[e] = silu_f(v[e]);
  if (V == 4) *reinterpret_cast<float4*>(px) = *reinterpret_cast<const float4*>(v);
  else px[0] = v[0];
}

template <typename TX>
__global__ void short_conv_tail_kernel(const TX* __restrict__ x, long long ldx, const float* __restrict__ in_bias, float* __restrict__ state,
                                       const int* __restrict__ runs, const int* __restrict__ pos, const int* __restrict__ slot,
                                       int n_runs, int C, int taps) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)n_runs * C) return;
  const int r = (int)(idx / C), c = (int)(idx % C);
  int first, n, p0, s;
  if (runs) { first = runs[4 * r]; n = runs[4 * r + 1]; p0 = runs[4 * r + 2]; s = runs[4 * r + 3]; }
  else { first = r; n = 1; p0 = pos[r]; s = slot[r]; }
  const int L = taps - 1;
  float* st = state + (long long)s * L * C + c;
  float nv[kMaxTaps];
  for (int i = 0; i < L; ++i) {
    const int q = p0 + n - L + i;                        // position whose input lands in entry i
    float v = 0.f;
    if (q >= p0) v = to_f32<TX>(x[(long long)(first + (q - p0)) * ldx + c]) + (in_bias ? in_bias[c] : 0.f);
    else if (q >= 0) v = st[(long long)(q - p0 + L) * C];
    nv[i] = v;
  }
  for (int i = 0; i < L; ++i) st[(long long)i * C] = nv[i];
}

// one warp per row of q / k / a, one thread per b
__global__ void __launch_bounds__(128)
delta_gates_kernel(float* __restrict__ q, long long ldq, float* __restrict__ k, long long ldk, float* __restrict__ a,
                   long long lda, float* __restrict__ b, long long ldb, const float* __restrict__ dt_bias,
                   const float* __restrict__ A_log, int G, int H, int D, int AD, float qscale, float unit_eps) {
  const int t = blockIdx.x;                               // AD: decays per head (D, or 1)
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const bool v4 = D % 4 == 0 && D <= 128 && ldq % 4 == 0 && ldk % 4 == 0 &&
                  !((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k)) & 15);
  for (int r = warp; r < 2 * G + (AD > 1 ? H : 0); r += nw) {
    if (r < 2 * G) {
      float* x = r < G ? q + (long long)t * ldq + (long long)r * D : k + (long long)t * ldk + (long long)(r - G) * D;
      if (v4) {                                           // a row is at most one 16-byte group per lane
        float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
        if (lane * 4 < D) u = *reinterpret_cast<const float4*>(x + lane * 4);
        const float sc = rsqrtf(warp_sum(u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w) + unit_eps) * (r < G ? qscale : 1.f);
        if (lane * 4 < D) *reinterpret_cast<float4*>(x + lane * 4) = make_float4(u.x * sc, u.y * sc, u.z * sc, u.w * sc);
        continue;
      }
      float ss = 0.f;
      for (int d = lane; d < D; d += 32) ss += x[d] * x[d];
      ss = warp_sum(ss);
      const float sc = rsqrtf(ss + unit_eps) * (r < G ? qscale : 1.f);
      for (int d = lane; d < D; d += 32) x[d] *= sc;
    } else {
      const int h = r - 2 * G;
      float* x = a + (long long)t * lda + (long long)h * AD;
      const float rate = expf(A_log[h]);
      for (int d = lane; d < AD; d += 32) {
        const float z = x[d] + dt_bias[h * AD + d];
        const float sp = z > 20.f ? z : log1pf(expf(z));
        x[d] = expf(-rate * sp);
      }
    }
  }
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    float* x = b + (long long)t * ldb + h;
    *x = 1.f / (1.f + expf(-*x));
    if (AD == 1) {
      float* y = a + (long long)t * lda + h;
      const float z = *y + dt_bias[h];
      *y = expf(-expf(A_log[h]) * (z > 20.f ? z : log1pf(expf(z))));
    }
  }
}

// out[s, t, c] = h[t, c] + (h' - h[t, c]) mu[s, c], h' the previous token's h: the row before inside a run, else `prev`
// [rows, W] (zeros at position 0). step_tail: every token is a run of its own, so the thread that read prev also replaces it.
template <typename T, int V>
__global__ void __launch_bounds__(256)
token_shift_kernel(const T* __restrict__ h, long long ldh, const float* __restrict__ mu, float* __restrict__ prev,
                   const int* __restrict__ pos, const int* __restrict__ slot, T* __restrict__ out, int tokens, int W, int S,
                   int step_tail) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int WV = W / V;
  if (idx >= (long long)tokens * WV) return;
  const int t = (int)(idx / WV), c = (int)(idx % WV) * V;
  const int p = pos[t], s = slot[t];
  float x[V], y[V];
  load_f32<V, T>(h + (long long)t * ldh + c, x);
#pragma unroll
  for (int e = 0; e < V; ++e) y[e] = 0.f;
  float* pr = prev + (long long)s * W + c;
  if (p > 0) {
    if (!step_tail && t > 0 && slot[t - 1] == s && pos[t - 1] == p - 1) load_f32<V, T>(h + (long long)(t - 1) * ldh + c, y);
    else load_f32<V, float>(pr, y);
  }
  if (step_tail) {
#pragma unroll
    for (int e = 0; e < V; ++e) pr[e] = x[e];
  }
#pragma unroll
  for (int e = 0; e < V; ++e) y[e] -= x[e];
  for (int i = 0; i < S; ++i) {
    float m[V], r[V];
    load_f32<V, float>(mu + (long long)i * W + c, m);
#pragma unroll
    for (int e = 0; e < V; ++e) r[e] = fmaf(y[e], m[e], x[e]);
    T* dst = out + ((long long)i * tokens + t) * W + c;
    if (V == 4 && sizeof(T) == 4) *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(r);
    else if (V == 4) *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(r[0], r[1 % V]), pack_bf16x2(r[V > 2 ? 2 : 0], r[V - 1]));
    else dst[0] = from_f32<T>(r[0]);
  }
}

constexpr int kScanChunk = 16;

__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16f(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// grid (runs, H, column blocks); block = NW warps; a warp covers 32 / LPC columns, lane = l * (32 / LPC) + jj. The chunk of
// tokens after the one being walked is already on its way into the other shared-memory buffer (cp.async), so the walk
// waits for global memory once per run, not once per chunk. `vec`: rows of q / k / g start on 16-byte boundaries.
template <int R, int MODE, int LPC>
__global__ void __launch_bounds__(128)
linear_scan_kernel(const float* __restrict__ q, long long ldq, const float* __restrict__ k, long long ldk,
                   const float* __restrict__ v, long long ldv, const float* __restrict__ g, long long ldg,
                   const float* __restrict__ beta, long long ldb, const float* __restrict__ decay, float* __restrict__ state,
                   const int* __restrict__ runs, const int* __restrict__ pos, const int* __restrict__ slot,
                   float* __restrict__ o, int H, int G, int D, int Dv, int act, int vec, int ones) {
  // MODE 2 reads its two per-token numbers through the pointers of mode 1's per-channel decays: g = a [T, H], beta = b [T, H];
  // MODE 3 likewise its decay and beta
  constexpr bool DELTA = MODE == 1 || MODE == 3;
  extern __shared__ __align__(16) float sm[];
  const int r_ = blockIdx.x, h = blockIdx.y;
  int first, n, p0, s;
  if (runs) { first = runs[4 * r_]; n = runs[4 * r_ + 1]; p0 = runs[4 * r_ + 2]; s = runs[4 * r_ + 3]; }
  else { first = r_; n = 1; p0 = pos[r_]; s = slot[r_]; }
  const int kvh = h / (H / G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  constexpr int cpw = 32 / LPC;                           // columns per warp
  const int l = lane / cpw, jj = lane % cpw;
  const int ncol = nw * cpw;                              // columns per CTA
  const int col0 = blockIdx.z * ncol;
  const int j = col0 + warp * cpw + jj;
  const bool live = j < Dv;
  const int row0 = l * R;
  constexpr int RP = R + 4;                               // a lane group's rows, padded so that the groups' 16-byte reads
  constexpr int DP = LPC * RP;                            // of one token fall into different banks
  auto at = [](int d) { return (d / R) * RP + d % R; };   // key channel d -> its place in a staged row
  const int ncp = (ncol + 3) & ~3;
  const int vcols = Dv - ones;                            // columns that come from v; column vcols, if any, is all ones
  const int per = kScanChunk * DP * (MODE == 1 ? 3 : 2) + kScanChunk * ncp + 2 * kScanChunk;  // floats per buffer
  auto KS = [&](int b) { return sm + b * per; };                                               // [chunk][DP]
  auto QS = [&](int b) { return sm + b * per + kScanChunk * DP; };
  auto GS = [&](int b) { return sm + b * per + 2 * kScanChunk * DP; };                         // MODE 1 only
  auto VS = [&](int b) { return sm + b * per + (MODE == 1 ? 3 : 2) * kScanChunk * DP; };       // [chunk][ncp]
  auto BS = [&](int b) { return VS(b) + kScanChunk * ncp; };                                   // [chunk]
  auto AS = [&](int b) { return VS(b) + kScanChunk * ncp + kScanChunk; };                      // [chunk], MODE 2 and 3 only
  float* os = sm + 2 * per;                               // [chunk][ncol][LPC]: per-lane parts of the read-outs of a chunk
  // padding rows (D <= d < DP) never arrive by copy: k = q = 0 (and a finite g) keep their state at zero
  if (LPC * R > D) {
    const int padw = LPC * R - D;
    for (int i = threadIdx.x; i < 2 * kScanChunk * padw; i += blockDim.x) {
      const int b = i / (kScanChunk * padw), r = i % (kScanChunk * padw);
      const int x = (r / padw) * DP + at(D + r % padw);
      KS(b)[x] = 0.f;
      QS(b)[x] = 0.f;
      if (MODE == 1) GS(b)[x] = 0.f;
    }
  }
  // the state rows of a thread as pairs: the walk runs on packed fp32 FMAs (two IEEE FMAs per instruction, same results)
  float2 S2[R / 2];
  float* sp = state + (((long long)s * H + h) * D) * Dv;
#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
    S2[i].x = (p0 > 0 && live && row0 + 2 * i < D) ? sp[(long long)(row0 + 2 * i) * Dv + j] : 0.f;
    S2[i].y = (p0 > 0 && live && row0 + 2 * i + 1 < D) ? sp[(long long)(row0 + 2 * i + 1) * Dv + j] : 0.f;
  }
  const float dec = MODE == 0 ? decay[h] : 0.f;

  auto stage = [&](int b, int c0) {
    const int cn = min(kScanChunk, n - c0);
    for (int tt = warp; tt < cn; tt += nw) {
      const long long tr = first + c0 + tt;
      const float* kr = k + tr * ldk + (long long)kvh * D;
      const float* qr = q + tr * ldq + (long long)kvh * D;
      const float* gr = MODE == 1 ? g + tr * ldg + (long long)h * D : nullptr;
      if (vec) {
        for (int d = lane * 4; d < D; d += 128) {
          cp_async16f(KS(b) + tt * DP + at(d), kr + d);
          cp_async16f(QS(b) + tt * DP + at(d), qr + d);
          if (MODE == 1) cp_async16f(GS(b) + tt * DP + at(d), gr + d);
        }
      } else {
        for (int d = lane; d < D; d += 32) {
          cp_async4(KS(b) + tt * DP + at(d), kr + d);
          cp_async4(QS(b) + tt * DP + at(d), qr + d);
          if (MODE == 1) cp_async4(GS(b) + tt * DP + at(d), gr + d);
        }
      }
      const float* vr = v + tr * ldv + (long long)h * vcols + col0;
      for (int cc = lane; cc < ncol && col0 + cc < Dv; cc += 32) {
        if (col0 + cc < vcols) cp_async4(VS(b) + tt * ncp + cc, vr + cc);
        else VS(b)[tt * ncp + cc] = 1.f;
      }
      if (MODE >= 1 && lane == 0) cp_async4(BS(b) + tt, beta + tr * ldb + h);
      if (MODE >= 2 && lane == 1) cp_async4(AS(b) + tt, g + tr * ldg + h);
    }
  };

  stage(0, 0);
  cp_commit();
  int buf = 0;
  for (int c0 = 0; c0 < n; c0 += kScanChunk, buf ^= 1) {
    const int cn = min(kScanChunk, n - c0);
    const bool more = c0 + kScanChunk < n;
    if (more) stage(buf ^ 1, c0 + kScanChunk);
    cp_commit();
    cp_wait<1>();
    __syncthreads();
    if (act) {
      for (int i = threadIdx.x; i < cn * DP; i += blockDim.x) { KS(buf)[i] = silu_f(KS(buf)[i]); QS(buf)[i] = silu_f(QS(buf)[i]); }
      for (int i = threadIdx.x; i < cn * ncp; i += blockDim.x) VS(buf)[i] = silu_f(VS(buf)[i]);
      __syncthreads();
    }
    const float* ks = KS(buf);
    const float* qs = QS(buf);
    const float* gs = GS(buf);
    const float* vs = VS(buf);
    const float* bs = BS(buf);
    const float* as = AS(buf);
    const float* vsp = vs + warp * cpw + jj;
    float* osp = os + (warp * cpw + jj) * LPC + l;
#pragma unroll 4
    for (int tt = 0; tt < cn; ++tt) {
      float2 kr[R / 2], qr[R / 2];
#pragma unroll
      for (int i = 0; i < R / 2; i += 2) {
        const float4 k4 = *reinterpret_cast<const float4*>(ks + tt * DP + l * RP + 2 * i);
        const float4 q4 = *reinterpret_cast<const float4*>(qs + tt * DP + l * RP + 2 * i);
        kr[i] = make_float2(k4.x, k4.y); kr[i + 1] = make_float2(k4.z, k4.w);
        qr[i] = make_float2(q4.x, q4.y); qr[i + 1] = make_float2(q4.z, q4.w);
      }
      const float vj = MODE == 2 ? vsp[tt * ncp] * bs[tt] : vsp[tt * ncp];
      float2 oa = make_float2(0.f, 0.f), ob = make_float2(0.f, 0.f);
      if (!DELTA) {
        const float dt_ = MODE == 2 ? as[tt] : dec;
        const float2 v2 = make_float2(vj, vj), dec2 = make_float2(dt_, dt_);
#pragma unroll
        for (int i = 0; i < R / 2; i += 2) {
          S2[i] = __ffma2_rn(dec2, S2[i], __fmul2_rn(kr[i], v2));
          S2[i + 1] = __ffma2_rn(dec2, S2[i + 1], __fmul2_rn(kr[i + 1], v2));
          oa = __ffma2_rn(S2[i], qr[i], oa);
          ob = __ffma2_rn(S2[i + 1], qr[i + 1], ob);
        }
      } else {
        float2 da = make_float2(0.f, 0.f), db = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < R / 2; i += 2) {
          const float a_ = MODE == 3 ? as[tt] : 0.f;
          const float4 g4 = MODE == 3 ? make_float4(a_, a_, a_, a_) : *reinterpret_cast<const float4*>(gs + tt * DP + l * RP + 2 * i);
          S2[i] = __fmul2_rn(S2[i], make_float2(g4.x, g4.y));
          S2[i + 1] = __fmul2_rn(S2[i + 1], make_float2(g4.z, g4.w));
          da = __ffma2_rn(S2[i], kr[i], da);
          db = __ffma2_rn(S2[i + 1], kr[i + 1], db);
        }
        float dot = (da.x + da.y) + (db.x + db.y);
#pragma unroll
        for (int x = cpw; x < 32; x <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, x);
        const float u = bs[tt] * (vj - dot);
        const float2 u2 = make_float2(u, u);
#pragma unroll
        for (int i = 0; i < R / 2; i += 2) {
          S2[i] = __ffma2_rn(kr[i], u2, S2[i]);
          S2[i + 1] = __ffma2_rn(kr[i + 1], u2, S2[i + 1]);
          oa = __ffma2_rn(S2[i], qr[i], oa);
          ob = __ffma2_rn(S2[i + 1], qr[i + 1], ob);
        }
      }
      const float o0 = oa.x + oa.y, o1 = ob.x + ob.y;
      // a token's read-out stays a per-lane part until the chunk is walked: nothing but the state (and, for the delta rule,
      // the reduced S^T k) sits between one token and the next
      osp[tt * ncol * LPC] = o0 + o1;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < cn * ncol; i += blockDim.x) {
      const int tt = i / ncol, cc = i - tt * ncol;
      float a = 0.f;
#pragma unroll
      for (int x = 0; x < LPC; ++x) a += os[i * LPC + x];
      if (col0 + cc < Dv) o[((long long)(first + c0 + tt) * H + h) * Dv + col0 + cc] = a;
    }
    __syncthreads();
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      if (row0 + 2 * i < D) sp[(long long)(row0 + 2 * i) * Dv + j] = S2[i].x;
      if (row0 + 2 * i + 1 < D) sp[(long long)(row0 + 2 * i + 1) * Dv + j] = S2[i].y;
    }
  }
}

// One warp per (run, head), a lane per token of a chunk of 32: the gates are formed in parallel and the maximum recurrence
// m_t = max(f_t + m_(t-1), i_t) is a warp scan over max-plus maps; the maximum is carried from chunk to chunk.
__global__ void __launch_bounds__(128)
mlstm_gates_kernel(const float* __restrict__ gi, long long ldi, const float* __restrict__ gf, long long ldf,
                   const float* __restrict__ bi, const float* __restrict__ bf, float cap, float* __restrict__ mstate,
                   const int* __restrict__ runs, const int* __restrict__ pos, const int* __restrict__ slot, int n_runs, int H,
                   float* __restrict__ a, float* __restrict__ b, float* __restrict__ e) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * 4 + warp;
  if (w >= (long long)n_runs * H) return;
  const int r = (int)(w / H), h = (int)(w % H);
  int first, n, p0, s;
  if (runs) { first = runs[4 * r]; n = runs[4 * r + 1]; p0 = runs[4 * r + 2]; s = runs[4 * r + 3]; }
  else { first = r; n = 1; p0 = pos[r]; s = slot[r]; }
  float m = p0 > 0 ? mstate[(long long)s * H + h] : 0.f;
  const float bih = bi[h], bfh = bf[h];
  // the next chunk's gate inputs are fetched while this one is walked
  float gin = 0.f, gfn = 0.f;
  if (lane < n) { gin = gi[(long long)(first + lane) * ldi + h]; gfn = gf[(long long)(first + lane) * ldf + h]; }
  for (int c0 = 0; c0 < n; c0 += 32) {
    const int cn = min(32, n - c0);
    const float gic = gin, gfc = gfn;
    if (c0 + 32 + lane < n) {
      gin = gi[(long long)(first + c0 + 32 + lane) * ldi + h];
      gfn = gf[(long long)(first + c0 + 32 + lane) * ldf + h];
    }
    float fv = 0.f, iv = 0.f;
    if (lane < cn) {
      iv = cap * tanhf((gic + bih) / cap);
      const float z = cap * tanhf((gfc + bfh) / cap);
      fv = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));        // log sigmoid(z)
    }
    // token j maps the running maximum x to max(x + f_j, i_j); two such maps compose to one of the same form,
    // (A1, B1) then (A2, B2) = (A1 + A2, max(B1 + A2, B2)), so the 32 tokens of a chunk are a warp scan of five steps
    // instead of 32 dependent ones. Lanes past the chunk hold the identity (0, -inf). How the sums are rounded does not
    // matter downstream: decay and input scale below are formed from the same maxima.
    float A = lane < cn ? fv : 0.f, B = lane < cn ? iv : -INFINITY;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float Ap = __shfl_up_sync(0xffffffffu, A, d), Bp = __shfl_up_sync(0xffffffffu, B, d);
      if (lane >= d) { B = fmaxf(Bp + A, B); A = Ap + A; }
    }
    const float mnew = fmaxf(m + A, B);
    float mprev = __shfl_up_sync(0xffffffffu, mnew, 1);
    if (lane == 0) mprev = m;
    if (lane < cn) {
      const long long t = first + c0 + lane;
      a[t * H + h] = expf(fv + mprev - mnew);
      b[t * H + h] = expf(iv - mnew);
      e[t * H + h] = expf(-mnew);
    }
    m = __shfl_sync(0xffffffffu, mnew, cn - 1);
  }
  if (lane == 0) mstate[(long long)s * H + h] = m;
}

// The same for runs of many tokens: a CTA of eight warps per (run, head) takes 256 tokens per round. Every warp scans its
// chunk of 32 without knowing the incoming maximum (the composite map of a chunk does not depend on it), leaves the
// chunk's composite in shared memory, and then walks the composites of the chunks before it (at most seven steps) to get
// its own incoming maximum.
__global__ void __launch_bounds__(256)
mlstm_gates_run_kernel(const float* __restrict__ gi, long long ldi, const float* __restrict__ gf, long long ldf,
                       const float* __restrict__ bi, const float* __restrict__ bf, float cap, float* __restrict__ mstate,
                       const int* __restrict__ runs, int H, float* __restrict__ a, float* __restrict__ b, float* __restrict__ e) {
  __shared__ float cA[8], cB[8];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.x / H, h = blockIdx.x - r * H;
  const int first = runs[4 * r], n = runs[4 * r + 1], p0 = runs[4 * r + 2], s = runs[4 * r + 3];
  float m = p0 > 0 ? mstate[(long long)s * H + h] : 0.f;
  const float bih = bi[h], bfh = bf[h];
  for (int c0 = 0; c0 < n; c0 += 256) {
    const int t0 = c0 + warp * 32;
    const int cn = max(0, min(32, n - t0));
    float fv = 0.f, iv = 0.f;
    if (lane < cn) {
      const long long t = first + t0 + lane;
      iv = cap * tanhf((gi[t * ldi + h] + bih) / cap);
      const float z = cap * tanhf((gf[t * ldf + h] + bfh) / cap);
      fv = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));        // log sigmoid(z)
    }
    float A = lane < cn ? fv : 0.f, B = lane < cn ? iv : -INFINITY;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float Ap = __shfl_up_sync(0xffffffffu, A, d), Bp = __shfl_up_sync(0xffffffffu, B, d);
      if (lane >= d) { B = fmaxf(Bp + A, B); A = Ap + A; }
    }
    if (lane == 31) { cA[warp] = A; cB[warp] = B; }
    __syncthreads();
    float min_ = m, mend = m;
#pragma unroll
    for (int w2 = 0; w2 < 8; ++w2) {
      if (w2 == warp) min_ = mend;
      mend = fmaxf(mend + cA[w2], cB[w2]);
    }
    const float mnew = fmaxf(min_ + A, B);
    float mprev = __shfl_up_sync(0xffffffffu, mnew, 1);
    if (lane == 0) mprev = min_;
    if (lane < cn) {
      const long long t = first + t0 + lane;
      a[t * H + h] = expf(fv + mprev - mnew);
      b[t * H + h] = expf(iv - mnew);
      e[t * H + h] = expf(-mnew);
    }
    m = mend;
    __syncthreads();
  }
  if (threadIdx.x == 0) mstate[(long long)s * H + h] = m;
}

__global__ void ssm_gates_kernel(const float* __restrict__ dt, long long ld, const float* __restrict__ dt_bias,
                                 const float* __restrict__ A_log, float* __restrict__ a, float* __restrict__ b, long long tokens,
                                 int H) {
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= tokens * H) return;
  const long long t = idx / H;
  const int h = (int)(idx - t * H);
  const float z = dt[t * ld + h] + dt_bias[h];
  const float sp = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));  // softplus without a threshold
  a[idx] = expf(-expf(A_log[h]) * sp);
  b[idx] = sp;
}

// One CTA per token; the row [N = H * Dv] lives in shared memory between the passes. o rows have `ocols` columns per head
// (Dv, or Dv + 1 when the scan carried a column of ones).
template <typename TO, typename TG>
__global__ void __launch_bounds__(256)
scan_readout_kernel(const float* __restrict__ o, int ocols, const float* __restrict__ e, float den_eps, float oscale,
                    const float* __restrict__ skip, const float* __restrict__ x, long long ldx,
                    const float* __restrict__ pre, long long ldpre, const TG* __restrict__ post, long long ldpost,
                    int post_silu, const float* __restrict__ w, int w_full, TO* __restrict__ out, int H, int Dv, int groups, float eps) {
  extern __shared__ float row[];                         // [N] + [groups]
  const long long t = blockIdx.x;
  const int N = H * Dv, GS = N / groups;
  float* gsum = row + N;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const float* orow = o + t * (long long)H * ocols;
  for (int c = threadIdx.x; c < N; c += blockDim.x) {
    const int h = c / Dv, d = c - h * Dv;
    float v = orow[h * ocols + d] * oscale;
    if (e) v = v / (fmaxf(fabsf(orow[h * ocols + Dv] * oscale), e[t * H + h]) + den_eps);
    if (skip) v = fmaf(skip[h], x[t * ldx + c], v);
    if (pre) { const float z = pre[t * ldpre + c]; v *= z / (1.f + expf(-z)); }
    row[c] = v;
  }
  __syncthreads();
  for (int g = warp; g < groups; g += nw) {
    float ss = 0.f;
    for (int i = lane; i < GS; i += 32) { const float v = row[g * GS + i]; ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    if (lane == 0) gsum[g] = 1.f / sqrtf(ss / (float)GS + eps);
  }
  __syncthreads();
  for (int c = threadIdx.x; c < N; c += blockDim.x) {
    float v = row[c] * gsum[c / GS] * w[w_full ? c : c % GS];
    if (post) { const float z = to_f32<TG>(post[t * ldpost + c]); v *= (post_silu ? z : 1.f) / (1.f + expf(-z)); }
    out[t * N + c] = from_f32<TO>(v);
  }
}
}  // namespace b200

B200_API int b200_short_conv_ex(const void* x, long long ldx, const float* w, const float* bias, float* state,
                                const int* pos, const int* slot, void* y, long long ldy, int tokens, int C, int taps, int act,
                                int residual, int step_tail, int x_dtype, int y_dtype, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  if (C <= 0 || taps < 1 || taps > kMaxTaps) return B200_ERR_BAD_SHAPE;
  if ((y_dtype != B200_DT_FP32 && y_dtype != B200_DT_BF16) || (x_dtype != B200_DT_FP32 && x_dtype != B200_DT_BF16))
    return B200_ERR_UNSUPPORTED;
  cudaStream_t st = (cudaStream_t)stream;
  const bool vec = C % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0 && !(reinterpret_cast<uintptr_t>(state) & 15) &&
                   !(reinterpret_cast<uintptr_t>(x) & (x_dtype == B200_DT_FP32 ? 15 : 7)) &&
                   !(reinterpret_cast<uintptr_t>(y) & (y_dtype == B200_DT_FP32 ? 15 : 7));
  const long long n = (long long)tokens * (vec ? C / 4 : C);
  const unsigned grid = (unsigned)((n + 255) / 256);
  if (!step_tail && taps <= 5) {
    const int TB = tokens >= 2048 ? 16 : (tokens >= 256 ? 4 : 1);
    const int per = 128 * (vec ? 4 : 1);
    const dim3 rgrid((C + per - 1) / per, (tokens + TB - 1) / TB);
    if (rgrid.y > 65535) return B200_ERR_TOO_LARGE;
#define CONVR(VV, TX, TY, TT)                                                                                                \
  short_conv_run_kernel<VV, TX, TY, TT><<<rgrid, 128, 0, st>>>((const TX*)x, ldx, w, bias, state, pos, slot, (TY*)y, ldy, tokens, C, act, \
                                                               residual, TB)
#define CONVR_T(VV, TX, TY)                                                                                                  \
  switch (taps) {                                                                                                            \
    case 1: CONVR(VV, TX, TY, 1); break; case 2: CONVR(VV, TX, TY, 2); break; case 3: CONVR(VV, TX, TY, 3); break;           \
    case 4: CONVR(VV, TX, TY, 4); break; default: CONVR(VV, TX, TY, 5); break;                                               \
  }
#define CONVR_Y(TX, TY) do { if (vec) { CONVR_T(4, TX, TY) } else { CONVR_T(1, TX, TY) } } while (0)
    if (x_dtype == B200_DT_FP32) { if (y_dtype == B200_DT_FP32) CONVR_Y(float, float); else CONVR_Y(float, __nv_bfloat16); }
    else { if (y_dtype == B200_DT_FP32) CONVR_Y(__nv_bfloat16, float); else CONVR_Y(__nv_bfloat16, __nv_bfloat16); }
#undef CONVR_Y
#undef CONVR_T
#undef CONVR
    B200_LAUNCH_CHECK();
    return 0;
  }
#define CONV(VV, TX, TY)                                                                                                     \
  short_conv_kernel<VV, TX, TY><<<grid, 256, 0, st>>>((const TX*)x, ldx, w, bias, state, pos, slot, (TY*)y, ldy, tokens, C, taps, act, \
                                                      residual, step_tail)
#define CONV_X(TX)                                                                                                           \
  do {                                                                                                                       \
    if (y_dtype == B200_DT_FP32) { if (vec) CONV(4, TX, float); else CONV(1, TX, float); }                                   \
    else { if (vec) CONV(4, TX, __nv_bfloat16); else CONV(1, TX, __nv_bfloat16); }                                           \
  } while (0)
  if (x_dtype == B200_DT_FP32) CONV_X(float); else CONV_X(__nv_bfloat16);
#undef CONV_X
#undef CONV
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_short_conv(const float* x, long long ldx, const float* w, const float* state, const int* pos, const int* slot,
                             float* y, long long ldy, int tokens, int C, int taps, int act, void* stream) {
  return b200_short_conv_ex(x, ldx, w, nullptr, const_cast<float*>(state), pos, slot, y, ldy, tokens, C, taps, act, 0, 0, B200_DT_FP32,
                            B200_DT_FP32, stream);
}

B200_API int b200_silu_rows(float* x, long long ld, long long rows, int cols, void* stream) {
  using namespace b200;
  if (rows <= 0 || cols <= 0) return 0;
  const bool vec = cols % 4 == 0 && ld % 4 == 0 && !(reinterpret_cast<uintptr_t>(x) & 15);
  const long long n = rows * (vec ? cols / 4 : cols);
  if (vec) silu_rows_kernel<4><<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, ld, rows, cols);
  else silu_rows_kernel<1><<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, ld, rows, cols);
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_short_conv_tail(const void* x, long long ldx, const float* in_bias, float* state, const int* runs, const int* pos,
                                  const int* slot, int n_runs, int C, int taps, int x_dtype, void* stream) {
  using namespace b200;
  if (n_runs <= 0 || taps <= 1) return 0;
  if (C <= 0 || taps > kMaxTaps) return B200_ERR_BAD_SHAPE;
  const long long n = (long long)n_runs * C;
  const unsigned grid = (unsigned)((n + 255) / 256);
  cudaStream_t st = (cudaStream_t)stream;
  if (x_dtype == B200_DT_FP32)
    short_conv_tail_kernel<float><<<grid, 256, 0, st>>>((const float*)x, ldx, in_bias, state, runs, pos, slot, n_runs, C, taps);
  else if (x_dtype == B200_DT_BF16)
    short_conv_tail_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>((const __nv_bfloat16*)x, ldx, in_bias, state, runs, pos, slot, n_runs, C, taps);
  else return B200_ERR_UNSUPPORTED;
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_delta_gates_ex(float* q, long long ldq, float* k, long long ldk, float* a, long long lda, float* b, long long ldb,
                                 const float* dt_bias, const float* A_log, int tokens, int G, int H, int D, int AD, float qscale,
                                 float unit_eps, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  if (AD != D && AD != 1) return B200_ERR_BAD_SHAPE;
  delta_gates_kernel<<<tokens, 128, 0, (cudaStream_t)stream>>>(q, ldq, k, ldk, a, lda, b, ldb, dt_bias, A_log, G, H, D, AD, qscale, unit_eps);
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_delta_gates(float* q, long long ldq, float* k, long long ldk, float* a, long long lda, float* b, long long ldb,
                              const float* dt_bias, const float* A_log, int tokens, int G, int H, int D, float qscale,
                              float unit_eps, void* stream) {
  return b200_delta_gates_ex(q, ldq, k, ldk, a, lda, b, ldb, dt_bias, A_log, tokens, G, H, D, D, qscale, unit_eps, stream);
}

B200_API int b200_token_shift(const void* h, long long ldh, const float* mu, float* prev, const int* pos, const int* slot, void* out,
                              int tokens, int W, int S, int step_tail, int dtype, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  if (W <= 0 || S <= 0) return B200_ERR_BAD_SHAPE;
  cudaStream_t st = (cudaStream_t)stream;
  const int es = dtype == B200_DT_FP32 ? 4 : 2;
  const bool vec = W % 4 == 0 && ldh % 4 == 0 && !((reinterpret_cast<uintptr_t>(mu) | reinterpret_cast<uintptr_t>(prev)) & 15) &&
                   !((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(out)) & (4 * es - 1));
  const long long n = (long long)tokens * (vec ? W / 4 : W);
  const unsigned grid = (unsigned)((n + 255) / 256);
#define SHIFT(TT, VV) token_shift_kernel<TT, VV><<<grid, 256, 0, st>>>((const TT*)h, ldh, mu, prev, pos, slot, (TT*)out, tokens, W, S, step_tail)
  if (dtype == B200_DT_FP32) { if (vec) SHIFT(float, 4); else SHIFT(float, 1); }
  else if (dtype == B200_DT_BF16) { if (vec) SHIFT(__nv_bfloat16, 4); else SHIFT(__nv_bfloat16, 1); }
  else return B200_ERR_UNSUPPORTED;
#undef SHIFT
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_linear_scan(const float* q, long long ldq, const float* k, long long ldk, const float* v, long long ldv,
                              const float* g, long long ldg, const float* beta, long long ldb, const float* decay, float* state,
                              const int* runs, const int* pos, const int* slot, int n_runs, float* o, int H, int G, int D, int Dv,
                              int mode, int act, int ones, void* stream) {
  using namespace b200;
  if (n_runs <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || Dv <= 0 || mode < 0 || mode > 3 || H > 65535 || ones < 0 || ones > 1 || Dv - ones < 1)
    return B200_ERR_BAD_SHAPE;
  // rows per thread R in {8, 16, 32}; lanes per column LPC = power of two with LPC * R >= D
  int R = D <= 8 ? 8 : (D <= 256 ? 16 : 32);
  int LPC = 1;
  while (LPC * R < D) LPC *= 2;
  if (LPC > 32) return B200_ERR_TOO_LARGE;
  const int cpw = 32 / LPC;
  int nw = 4;
  while (nw > 1 && (nw - 1) * cpw >= Dv) --nw;            // no warp without columns
  const int ncol = nw * cpw;
  const int zb = (Dv + ncol - 1) / ncol;
  const int DP = LPC * (R + 4);
  const int ncp = (ncol + 3) & ~3;
  const size_t smem = (2 * ((size_t)kScanChunk * DP * (mode == 1 ? 3 : 2) + (size_t)kScanChunk * ncp + 2 * kScanChunk) +
                       (size_t)kScanChunk * ncol * LPC) * 4;
  if (smem > 200 * 1024) return B200_ERR_TOO_LARGE;
  auto al = [](const void* p_, long long ld) { return !(reinterpret_cast<uintptr_t>(p_) & 15) && ld % 4 == 0; };
  const int vec = D % 4 == 0 && al(q, ldq) && al(k, ldk) && (mode != 1 || al(g, ldg));
  dim3 grid(n_runs, H, zb);
  cudaStream_t st = (cudaStream_t)stream;
#define SCAN_K(RR, MM, LL)                                                                                                 \
  do {                                                                                                                     \
    auto kern = linear_scan_kernel<RR, MM, LL>;                                                                            \
    if (smem > 48 * 1024) B200_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));  \
    kern<<<grid, nw * 32, smem, st>>>(q, ldq, k, ldk, v, ldv, g, ldg, beta, ldb, decay, state, runs, pos, slot, o, H, G, D, Dv, act, vec, ones); \
  } while (0)
#define SCAN(RR, LL)                                                                                                       \
  do {                                                                                                                     \
    if (mode == 0) SCAN_K(RR, 0, LL); else if (mode == 1) SCAN_K(RR, 1, LL); else if (mode == 2) SCAN_K(RR, 2, LL);        \
    else SCAN_K(RR, 3, LL);                                                                                                \
  } while (0)
  if (R == 8) SCAN(8, 1);
  else if (R == 16) {
    if (LPC == 1) SCAN(16, 1); else if (LPC == 2) SCAN(16, 2); else if (LPC == 4) SCAN(16, 4); else if (LPC == 8) SCAN(16, 8); else SCAN(16, 16);
  } else {
    if (LPC == 16) SCAN(32, 16); else SCAN(32, 32);
  }
#undef SCAN
#undef SCAN_K
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_mlstm_gates(const float* gi, long long ldi, const float* gf, long long ldf, const float* bi, const float* bf,
                              float cap, float* mstate, const int* runs, const int* pos, const int* slot, int n_runs, int H,
                              float* a, float* b, float* e, void* stream) {
  using namespace b200;
  if (n_runs <= 0) return 0;
  if (H <= 0 || !(cap > 0.f)) return B200_ERR_BAD_SHAPE;
  const long long warps = (long long)n_runs * H;
  if (runs) {                                              // pieces of prompts (and the single tokens beside them)
    if (warps > 0x7fffffffLL) return B200_ERR_TOO_LARGE;
    mlstm_gates_run_kernel<<<(unsigned)warps, 256, 0, (cudaStream_t)stream>>>(gi, ldi, gf, ldf, bi, bf, cap, mstate, runs, H, a, b, e);
    B200_LAUNCH_CHECK();
    return 0;
  }
  mlstm_gates_kernel<<<(unsigned)((warps + 3) / 4), 128, 0, (cudaStream_t)stream>>>(gi, ldi, gf, ldf, bi, bf, cap, mstate, runs, pos,
                                                                                    slot, n_runs, H, a, b, e);
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_ssm_gates(const float* dt, long long ld, const float* dt_bias, const float* A_log, float* a, float* b,
                            long long tokens, int H, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  if (H <= 0) return B200_ERR_BAD_SHAPE;
  const long long n = tokens * H;
  ssm_gates_kernel<<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(dt, ld, dt_bias, A_log, a, b, tokens, H);
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_scan_readout(const float* o, int ocols, const float* e, float den_eps, float oscale, const float* skip,
                               const float* x, long long ldx, const float* pre, long long ldpre, const void* post,
                               long long ldpost, int post_silu, int post_dtype, const float* w, int w_full, void* out, long long tokens,
                               int H, int Dv, int groups, float eps, int out_dtype, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  if (H <= 0 || Dv <= 0 || groups <= 0 || (H * Dv) % groups || ocols < Dv || (e && ocols < Dv + 1) || (skip && !x))
    return B200_ERR_BAD_SHAPE;
  const size_t smem = ((size_t)H * Dv + groups) * sizeof(float);
  if (smem > 200 * 1024) return B200_ERR_TOO_LARGE;
  cudaStream_t st = (cudaStream_t)stream;
#define READOUT(TO, TG)                                                                                                        \
  do {                                                                                                                       \
    auto kern = scan_readout_kernel<TO, TG>;                                                                                 \
    if (smem > 48 * 1024) B200_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));    \
    kern<<<(unsigned)tokens, 256, smem, st>>>(o, ocols, e, den_eps, oscale, skip, x, ldx, pre, ldpre, (const TG*)post, ldpost, post_silu, w, w_full,  \
                                              (TO*)out, H, Dv, groups, eps);                                                 \
  } while (0)
  const bool gate16 = post && post_dtype == B200_DT_BF16;
  if (gate16 && out_dtype == B200_DT_BF16) READOUT(__nv_bfloat16, __nv_bfloat16);
  else if (gate16) return B200_ERR_UNSUPPORTED;
  else if (out_dtype == B200_DT_FP32) READOUT(float, float);
  else if (out_dtype == B200_DT_BF16) READOUT(__nv_bfloat16, float);
  else return B200_ERR_UNSUPPORTED;
#undef READOUT
  B200_LAUNCH_CHECK();
  return 0;
}
