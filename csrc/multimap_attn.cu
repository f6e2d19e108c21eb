// Multi-map attention over the paged KV cache: M attention maps per head (each with its own query and key rows, all over the
// same values), a sliding window that keeps the first tokens of the sequence, and an optional differential combination.
//
//   keys    cache K [blocks, G * M, block_size, D]   (key head g, map m at row g * M + m; normed and rotated when stored)
//   values  cache V [blocks, G,     block_size, Dv]  (Dv need not equal D)
//   token t (position p of cache row slot[t]) sees key j of its row if j <= p and (p - j < window or j < keep_first);
//   window <= 0 means every j <= p; opts.chunk > 0 (instead of a window): only keys of p's own chunk, j / chunk == p / chunk.
//   a_m = softmax_j(scale q_{h,m} . k_{g,m,j}) V_g        g = h / (H / G)
//   M = 2, combine:  o = a_0 - lambda a_1 ;  o <- o / sqrt(mean(o^2) + eps) * post      (differential attention)
//   otherwise:       o = a_0 post (M = 1)
//   b200_attn_opts (one map, every field optional): scores pass cap tanh(s / cap) before the softmax; a number per head whose
//   exponential joins the softmax's denominator (a sink: no key, no value); o_h times sigmoid(gate[t, h]).
//
// b200_qkv_store           bias, per-(head, map) RMS norm with a weight over D (or none), rotary on the first `rot` dims in the split
//                          layout (dim i pairs with i + rot/2), values mixed with those another layer cached for the same token;
//                          q -> q_out in the cache dtype, k and v -> their pages. b200_qknorm_rope_store: its fp32 subset.
// b200_conv_qknorm_store   what stands in front of one-map attention whose projections pass a short causal convolution: bias,
//                          convolution over time on every channel of q | k | v (inputs before the run come from a carried tail),
//                          per-row RMS norm without a weight (v optional), q times a factor that grows with the position.
// b200_multimap_attn       per-token attention in fp32 arithmetic over a 16-bit or 32-bit cache; prompt pieces and decoded
//                          tokens take the same path: a vector kernel (16-byte row chunks, the heads of a KV group share the
//                          K/V reads, `nsplit` key ranges + a merge kernel for few tokens with many keys) and a scalar one
//                          (a warp per (token, head)) for row sizes that are not whole chunks.
#include "common.cuh"
#include "mma_sync.cuh"

#include <type_traits>
#include "../include/b200_ops.h"

#define B200_DISPATCH_T(dtype, ...)                                   \
  if (dtype == B200_DT_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
  else if (dtype == B200_DT_FP16) { using T = __half; __VA_ARGS__; }   \
  else if (dtype == B200_DT_FP32) { using T = float; __VA_ARGS__; }    \
  else return B200_ERR_UNSUPPORTED;

namespace b200 {

// proj [tokens, ld]: q rows (QR = H * M of D) at column 0, then (has_kv) k rows (KR = G * M of D) and v (G rows of Dv). A warp
// owns one of these rows over TB consecutive tokens. A row is walked as pairs: (i, i + rot / 2) inside the rotated part and
// (i, i + half of the rest) behind it, so every lane has both members of the pairs it turns; V pairs lie next to each other,
// a lane owns up to NI groups of them, their biases and norm weights stay in registers. Rows of v (and of a layer without
// rotation) are one unrotated part.
struct QkvStoreArgs {
  const void* proj; long long ld;
  const float *bias, *wq, *wk;                           // bias [QR D + KR D + G Dv] or NULL; wq NULL: rows are not normed
  const float *cs, *sn;                                  // [max_pos, rot / 2]
  const int *pos, *slot, *table;
  void *q_out, *ck, *cv;
  const void* v_first; const float* v_lambda;            // v <- (1 - lambda) v + lambda v_first at the token's place in that pool
  int max_blocks, tokens, QR, KR, G, D, Dv, rot, block_size, has_kv, TB;
  float eps;
};

template <typename TX, int V> __device__ __forceinline__ void load_v(const TX* p, float (&v)[V]) {
  if (V == 2 && std::is_same<TX, __nv_bfloat16>::value) {
    const float2 f = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p));
    v[0] = f.x; v[V - 1] = f.y;
  } else if (V == 2 && sizeof(TX) == 4) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[V - 1] = f.y;
  } else {
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = to_f32<TX>(p[e]);
  }
}
template <typename T, int V> __device__ __forceinline__ void store_v(T* p, const float (&v)[V]) {
  if (V == 2 && std::is_same<T, __nv_bfloat16>::value) *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v[0], v[V - 1]);
  else if (V == 2 && sizeof(T) == 4) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[V - 1]);
  else {
#pragma unroll
    for (int e = 0; e < V; ++e) p[e] = from_f32<T>(v[e]);
  }
}

template <typename TX, typename T, int V, int NI>
__global__ void __launch_bounds__(128)
qkv_store_kernel(const QkvStoreArgs a) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.y * 4 + warp;
  if (r >= a.QR + (a.has_kv ? a.KR + a.G : 0)) return;
  const bool is_q = r < a.QR, is_v = r >= a.QR + a.KR;
  const int RS = is_v ? a.Dv : a.D;
  const int col0 = is_v ? (a.QR + a.KR) * a.D + (r - a.QR - a.KR) * a.Dv : r * a.D;
  const int hr = is_v ? 0 : a.rot / 2;
  const int ph = (RS - 2 * hr + 1) / 2;                  // pairs behind the rotated part
  const float* w = is_v || !a.wq ? nullptr : (is_q ? a.wq : a.wk);
  int i0[NI], i1[NI];                                    // first member of a group of pairs, and how far the second lies; < 0: none
  float b0[NI][V], b1[NI][V], w0[NI][V], w1[NI][V];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int x = (lane + 32 * i) * V;
    if (x < hr) { i0[i] = x; i1[i] = x + hr; }
    else if (x < hr + ph) { i0[i] = x + hr; i1[i] = x + hr + ph < RS ? x + hr + ph : -1; }
    else i0[i] = i1[i] = -1;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      b0[i][e] = a.bias && i0[i] >= 0 ? a.bias[col0 + i0[i] + e] : 0.f;
      b1[i][e] = a.bias && i1[i] >= 0 ? a.bias[col0 + i1[i] + e] : 0.f;
      w0[i][e] = w && i0[i] >= 0 ? w[i0[i] + e] : 1.f;
      w1[i][e] = w && i1[i] >= 0 ? w[i1[i] + e] : 1.f;
    }
  }
  const float lam = is_v && a.v_first ? a.v_lambda[0] : 0.f;
  const int t0 = blockIdx.x * a.TB, t1 = min(a.tokens, t0 + a.TB);
  for (int t = t0; t < t1; ++t) {
    const int p = a.pos[t];
    const TX* src = reinterpret_cast<const TX*>(a.proj) + (long long)t * a.ld + col0;
    float x0[NI][V], x1[NI][V], ss = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
#pragma unroll
      for (int e = 0; e < V; ++e) x0[i][e] = x1[i][e] = 0.f;
      if (i0[i] >= 0) load_v<TX, V>(src + i0[i], x0[i]);
      if (i1[i] >= 0) load_v<TX, V>(src + i1[i], x1[i]);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        x0[i][e] += b0[i][e];
        x1[i][e] += b1[i][e];
        ss = fmaf(x0[i][e], x0[i][e], ss);
        ss = fmaf(x1[i][e], x1[i][e], ss);
      }
    }
    if (w) {
      const float f = rsqrtf(warp_sum(ss) / RS + a.eps);
#pragma unroll
      for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int e = 0; e < V; ++e) { x0[i][e] *= f * w0[i][e]; x1[i][e] *= f * w1[i][e]; }
    }
    T* dst;
    long long place = 0;
    if (is_q) dst = reinterpret_cast<T*>(a.q_out) + ((long long)t * a.QR + r) * a.D;
    else {
      const long long blk = a.table[(long long)a.slot[t] * a.max_blocks + p / a.block_size];
      const int off = p % a.block_size;
      if (is_v) place = ((blk * a.G + (r - a.QR - a.KR)) * a.block_size + off) * a.Dv;
      else place = ((blk * a.KR + (r - a.QR)) * a.block_size + off) * a.D;
      dst = reinterpret_cast<T*>(is_v ? a.cv : a.ck) + place;
    }
    const float* c = a.cs + (long long)p * hr;
    const float* s = a.sn + (long long)p * hr;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int x = (lane + 32 * i) * V;
      if (x < hr) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const float u = x0[i][e], v = x1[i][e], cc = c[x + e], sn = s[x + e];
          x0[i][e] = u * cc - v * sn;
          x1[i][e] = v * cc + u * sn;
        }
      } else if (is_v && a.v_first) {
        const T* vf = reinterpret_cast<const T*>(a.v_first) + place;
        float f0[V], f1[V];
#pragma unroll
        for (int e = 0; e < V; ++e) f0[e] = f1[e] = 0.f;
        if (i0[i] >= 0) load_v<T, V>(vf + i0[i], f0);
        if (i1[i] >= 0) load_v<T, V>(vf + i1[i], f1);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          x0[i][e] = (1.f - lam) * x0[i][e] + lam * f0[e];
          x1[i][e] = (1.f - lam) * x1[i][e] + lam * f1[e];
        }
      }
      if (i0[i] >= 0) store_v<T, V>(dst + i0[i], x0[i]);
      if (i1[i] >= 0) store_v<T, V>(dst + i1[i], x1[i]);
    }
  }
}

// proj [tokens, ld] = q (H rows of D) | k (G rows of D) | v (G rows of Dv). A warp owns one of these rows over TB consecutive
// tokens, every lane up to VI pairs (V = 2) or single channels; the last taps - 1 inputs of a channel stay in registers from
// token to token and are fetched anew (from proj, the tail, or zeros) where a run starts inside the block.
// TAPS: the convolution's taps at compile time.
constexpr int kConvMaxTaps = 5;
template <typename TX, typename T, int TAPS, int V, int VI>
__global__ void __launch_bounds__(128)
conv_qknorm_store_kernel(const TX* __restrict__ proj, long long ld, const float* __restrict__ bias, const float* __restrict__ w,
                         const float* __restrict__ tail, const int* __restrict__ pos, const int* __restrict__ slot,
                         const int* __restrict__ table, int max_blocks, T* __restrict__ q_out, T* __restrict__ ck, T* __restrict__ cv,
                         int tokens, int H, int G, int D, int Dv, int block_size, float eps, float temp_coef, float temp_every,
                         int norm_qk, int norm_v, int TB) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.y * 4 + warp;
  if (r >= H + 2 * G) return;
  const bool is_v = r >= H + G;
  const int RS = is_v ? Dv : D;
  const int col0 = is_v ? (H + G) * D + (r - H - G) * Dv : r * D;
  const int C = (H + G) * D + G * Dv;
  constexpr int L = TAPS - 1;
  float wt[VI][V][TAPS], hist[VI][V][L > 0 ? L : 1], b[VI][V];
#pragma unroll
  for (int i = 0; i < VI; ++i)
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const int c = (lane + 32 * i) * V + e;
      b[i][e] = (bias && c < RS) ? bias[col0 + c] : 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) wt[i][e][j] = c < RS ? w[(long long)(col0 + c) * TAPS + j] : 0.f;
#pragma unroll
      for (int j = 0; j < L; ++j) hist[i][e][j] = 0.f;
    }
  auto load = [&](int t, int i, float (&v)[V]) {           // the biased inputs of token t
    const int c = (lane + 32 * i) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = 0.f;
    if (c < RS) {
      const TX* p = proj + (long long)t * ld + col0 + c;
      if (V == 2 && sizeof(TX) == 2) {
        const float2 f = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p));
        v[0] = f.x; v[V - 1] = f.y;
      } else if (V == 2) {
        const float2 f = *reinterpret_cast<const float2*>(p);
        v[0] = f.x; v[V - 1] = f.y;
      } else v[0] = to_f32<TX>(p[0]);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += b[i][e];
    }
  };
  const int t0 = blockIdx.x * TB, t1 = min(tokens, t0 + TB);
  int ps = -1, pp = -2;
  for (int t = t0; t < t1; ++t) {
    const int p = pos[t], s = slot[t];
    if (L > 0 && !(s == ps && p == pp + 1)) {              // not the token after the last one: fetch what lies before it
      int nb = 0;
      while (nb < L && t - nb - 1 >= 0 && slot[t - nb - 1] == s && pos[t - nb - 1] == p - nb - 1) ++nb;
#pragma unroll
      for (int d = 1; d <= L; ++d)                         // d tokens back -> hist[L - d]
#pragma unroll
        for (int i = 0; i < VI; ++i) {
          float v[V];
#pragma unroll
          for (int e = 0; e < V; ++e) v[e] = 0.f;
          if (p - d >= 0) {
            if (d <= nb) load(t - d, i, v);
            else {
#pragma unroll
              for (int e = 0; e < V; ++e) {
                const int c = (lane + 32 * i) * V + e;
                if (c < RS) v[e] = tail[((long long)s * L + (L - (d - nb))) * C + col0 + c];
              }
            }
          }
#pragma unroll
          for (int e = 0; e < V; ++e) hist[i][e][L > 0 ? L - d : 0] = v[e];
        }
    }
    ps = s; pp = p;
    float y[VI][V], ss = 0.f;
#pragma unroll
    for (int i = 0; i < VI; ++i) {
      float v[V];
      load(t, i, v);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float a = 0.f;
#pragma unroll
        for (int j = 0; j < L; ++j) a = fmaf(wt[i][e][j], hist[i][e][j], a);
        a = fmaf(wt[i][e][TAPS - 1], v[e], a);
#pragma unroll
        for (int j = 0; j + 1 < L; ++j) hist[i][e][j] = hist[i][e][j + 1];
        if (L > 0) hist[i][e][L > 0 ? L - 1 : 0] = v[e];
        y[i][e] = a;
        ss = fmaf(a, a, ss);
      }
    }
    float f = 1.f;
    if (is_v ? norm_v : norm_qk) f = rsqrtf(warp_sum(ss) / RS + eps);
    if (r < H && temp_coef != 0.f) f *= 1.f + temp_coef * logf((float)floor((double)(p + 1) / (double)temp_every) + 1.f);
    T* dst;
    if (r < H) dst = q_out + ((long long)t * H + r) * D;
    else {
      const long long blk = table[(long long)s * max_blocks + p / block_size];
      const int off = p % block_size;
      dst = is_v ? cv + ((blk * G + (r - H - G)) * block_size + off) * Dv : ck + ((blk * G + (r - H)) * block_size + off) * D;
    }
#pragma unroll
    for (int i = 0; i < VI; ++i) {
      const int c = (lane + 32 * i) * V;
      if (c >= RS) continue;
      if (V == 2 && sizeof(T) == 2) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(y[i][0] * f, y[i][V - 1] * f);
      else if (V == 2) *reinterpret_cast<float2*>(dst + c) = make_float2(y[i][0] * f, y[i][V - 1] * f);
      else dst[c] = from_f32<T>(y[i][0] * f);
    }
  }
}

constexpr int kMaxDv = 256;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
// the first key position p sees besides kept ones: the window's lower edge, or the start of p's chunk
__device__ __forceinline__ int first_seen(int p, int window, int chunk) {
  if (chunk > 0) return p / chunk * chunk;
  return window > 0 && p + 1 - window > 0 ? p + 1 - window : 0;
}
template <typename T> __device__ __forceinline__ float capped_tanh(float x) { return tanh_ex2(x); }
template <> __device__ __forceinline__ float capped_tanh<float>(float x) { return tanhf(x); }
constexpr int kAcc = kMaxDv / 32;
constexpr int kMaxMaps = 2;

template <typename T>
__device__ __forceinline__ float dot_qk(const float* __restrict__ q, const T* __restrict__ k, int D) {
  float acc = 0.f;
  for (int d = 0; d < D; ++d) acc = fmaf(q[d], to_f32<T>(k[d]), acc);
  return acc;
}
template <>
__device__ __forceinline__ float dot_qk<__nv_bfloat16>(const float* __restrict__ q, const __nv_bfloat16* __restrict__ k, int D) {
  float acc = 0.f;
  if ((D & 7) == 0) {
    for (int d = 0; d < D; d += 8) {
      const uint4 raw = *reinterpret_cast<const uint4*>(k + d);
      const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = unpack_bf16x2(w[j]);
        acc = fmaf(q[d + 2 * j], f.x, acc);
        acc = fmaf(q[d + 2 * j + 1], f.y, acc);
      }
    }
  } else {
    for (int d = 0; d < D; ++d) acc = fmaf(q[d], __bfloat162float(k[d]), acc);
  }
  return acc;
}

template <typename T>
__global__ void __launch_bounds__(128)
multimap_attn_kernel(const T* __restrict__ q, const T* __restrict__ ck, const T* __restrict__ cv, const int* __restrict__ pos,
                     const int* __restrict__ slot, const int* __restrict__ table, int max_blocks, T* __restrict__ out, long long ldo, int tokens,
                     int H, int G, int M, int D, int Dv, int block_size, float scale, int window, int keep_first, int combine,
                     float lambda, float post, float eps, const b200_attn_opts opt) {
  extern __shared__ float qs[];                          // [warps, D]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const long long item = (long long)blockIdx.x * nw + warp;          // (token, head)
  if (item >= (long long)tokens * H) return;
  const int t = (int)(item / H), h = (int)(item % H);
  const int g = h / (H / G);
  const int p = pos[t];
  const int* trow = table + (long long)slot[t] * max_blocks;
  const int lo = first_seen(p, window, opt.chunk);
  const int n1 = window > 0 ? min(max(keep_first, 0), lo) : 0;       // kept first tokens that the window no longer covers
  const int total = n1 + (p + 1 - lo);
  float* myq = qs + warp * D;
  float res[kAcc];
#pragma unroll
  for (int i = 0; i < kAcc; ++i) res[i] = 0.f;
  for (int m = 0; m < M; ++m) {
    const T* qr = q + (((long long)t * H + h) * M + m) * D;
    __syncwarp();
    for (int d = lane; d < D; d += 32) myq[d] = to_f32<T>(qr[d]);
    __syncwarp();
    float mx = -INFINITY, l = 0.f;
    float acc[kAcc];
#pragma unroll
    for (int i = 0; i < kAcc; ++i) acc[i] = 0.f;
    const int kh = g * M + m;
    for (int i0 = 0; i0 < total; i0 += 32) {
      const int i = i0 + lane;
      const bool valid = i < total;
      long long voff = 0;
      float sc = -INFINITY;
      if (valid) {
        const int kp = i < n1 ? i : lo + (i - n1);
        const int blk = trow[kp / block_size];
        const int off = kp % block_size;
        sc = dot_qk<T>(myq, ck + (((long long)blk * G * M + kh) * block_size + off) * D, D) * scale;
        if (opt.softcap > 0.f) sc = opt.softcap * capped_tanh<T>(sc / opt.softcap);
        voff = (((long long)blk * G + g) * block_size + off) * Dv;
      }
      const float m_new = fmaxf(mx, warp_max(sc));
      const float pj = valid ? expf(sc - m_new) : 0.f;
      const float resc = (mx == -INFINITY) ? 0.f : expf(mx - m_new);
      l = l * resc + warp_sum(pj);
      mx = m_new;
#pragma unroll
      for (int a = 0; a < kAcc; ++a) acc[a] *= resc;
      const int nk = min(32, total - i0);
      for (int j = 0; j < nk; ++j) {
        const float w = __shfl_sync(0xffffffffu, pj, j);
        const long long ro = __shfl_sync(0xffffffffu, voff, j);
        const T* vr = cv + ro;
#pragma unroll
        for (int a = 0; a < kAcc; ++a) {
          const int d = lane + 32 * a;
          if (d < Dv) acc[a] = fmaf(w, to_f32<T>(vr[d]), acc[a]);
        }
      }
    }
    if (opt.sink) l += expf(opt.sink[h] - mx);
    const float inv = l > 0.f ? 1.f / l : 0.f;
    const float coef = (m == 0) ? 1.f : -lambda;
#pragma unroll
    for (int a = 0; a < kAcc; ++a) res[a] = fmaf(coef, acc[a] * inv, res[a]);
  }
  float mult = post;
  if (combine) {
    float ss = 0.f;
#pragma unroll
    for (int a = 0; a < kAcc; ++a) ss += (lane + 32 * a < Dv) ? res[a] * res[a] : 0.f;
    ss = warp_sum(ss);
    mult = rsqrtf(ss / Dv + eps) * post;
  }
  if (opt.gate) mult *= sigmoid_f(opt.gate[(long long)t * opt.ld_gate + h]);
  T* orow = out + (long long)t * ldo + (long long)h * Dv;
#pragma unroll
  for (int a = 0; a < kAcc; ++a) {
    const int d = lane + 32 * a;
    if (d < Dv) orow[d] = from_f32<T>(res[a] * mult);
  }
}
// Vector variant (D and Dv whole 16-byte chunks, at most 32 chunks each): a CTA owns one token, up to HB query heads of one
// KV group, ONE map and one range of the visible keys (blockIdx.z = range * M + map). A lane is (key sub-index, chunk): the
// CP lanes of a group read the key row of the map and the value row of one key with one 16-byte load each; scores are
// reduced over the group's lanes and every lane keeps its own running (max, sum, acc) per head — nothing crosses groups
// inside the loop. Groups are merged by shuffles at the end, the four warps through shared memory. With one map and one
// range the result is written directly; otherwise (max, sum, acc) go to `part` [tokens, H, M, nsplit, Dv + 2] and
// multimap_attn_merge_kernel merges ranges and maps.
// VC: value chunks per lane (2 when the value rows are wider than the key rows: a group then has only as many lanes as a key
// row has chunks, covers twice the keys per instruction, and every lane accumulates chunks c and c + CP of the values)
template <typename T, int HB, int VC>
__global__ void __launch_bounds__(128, 4)               // four CTAs per SM: a decode batch of 64 x 4 groups x 2 maps is one wave
multimap_attn_vec_kernel(const T* __restrict__ q, const T* __restrict__ ck, const T* __restrict__ cv, const int* __restrict__ pos,
                         const int* __restrict__ slot, const int* __restrict__ table, int max_blocks, T* __restrict__ out, long long ldo,
                         float* __restrict__ part, int H, int G, int M, int D, int Dv, int bs_log2, float scale, int window,
                         int keep_first, int nsplit, float post, int CP, int CPK, int CPV, const b200_attn_opts opt) {
  constexpr int E = 16 / sizeof(T);
  extern __shared__ float sm[];                          // [4 warps][HB][Dv + 2]
  const int t = blockIdx.x;
  const int rep = H / G;
  const int passes = (rep + HB - 1) / HB;
  const int g = blockIdx.y / passes;
  const int h0 = g * rep + (blockIdx.y % passes) * HB;
  const int nh = min(HB, g * rep + rep - h0);
  const int split = blockIdx.z / M, m = blockIdx.z % M;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int KPI = 32 / CP;
  const int kk = lane / CP, c = lane % CP;
  const bool liveK = c < CPK;
  bool liveV[VC];
#pragma unroll
  for (int x = 0; x < VC; ++x) liveV[x] = c + x * CP < CPV;
  const int p = pos[t];
  const int* trow = table + (long long)slot[t] * max_blocks;
  const int lo = first_seen(p, window, opt.chunk);
  const int n1 = window > 0 ? min(max(keep_first, 0), lo) : 0;
  const int total = n1 + (p + 1 - lo);
  int i_lo = 0, i_hi = total;
  if (nsplit > 1) {
    const int chunk = ((total + nsplit - 1) / nsplit + 31) / 32 * 32;
    i_lo = split * chunk;
    i_hi = min(total, i_lo + chunk);
  }
  // scores are kept in units of log 2 (scale * log2(e) is folded into q): one ex2 per exponential; the merge kernel reads
  // the recorded maxima in the same units
  // (with a cap: q . k scale / cap leaves the product, and cap log2(e) multiplies its tanh)
  const bool capped = opt.softcap > 0.f;
  const float sl2 = capped ? scale / opt.softcap : scale * kLog2e;
  const float cap2 = opt.softcap * kLog2e;
  float qv[HB][E], acc[HB][VC][E], mx[HB], l[HB];
#pragma unroll
  for (int hh = 0; hh < HB; ++hh) {
    mx[hh] = -INFINITY;
    l[hh] = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) {
#pragma unroll
      for (int x = 0; x < VC; ++x) acc[hh][x][e] = 0.f;
      qv[hh][e] = (liveK && hh < nh) ? to_f32<T>(q[(((long long)t * H + h0 + hh) * M + m) * D + c * E + e]) * sl2 : 0.f;
    }
  }
  const int bs_mask = (1 << bs_log2) - 1;
  const int stride = 4 * KPI;
  constexpr int U = HB >= 4 ? 2 : 4;
  for (int ib = i_lo; ib < i_hi; ib += stride * U) {
    uint4 kr[U], vr[U][VC];
    bool valid[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = ib + u * stride + warp * KPI + kk;
      valid[u] = i < i_hi;
      kr[u] = make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int x = 0; x < VC; ++x) vr[u][x] = make_uint4(0, 0, 0, 0);
      if (valid[u]) {
        const int kp = i < n1 ? i : lo + (i - n1);
        const long long blk = trow[kp >> bs_log2];
        const int off = kp & bs_mask;
        if (liveK) kr[u] = *reinterpret_cast<const uint4*>(ck + ((((blk * G + g) * M + m) << bs_log2) + off) * D + c * E);
#pragma unroll
        for (int x = 0; x < VC; ++x)
          if (liveV[x]) vr[u][x] = *reinterpret_cast<const uint4*>(cv + ((((blk * G) + g) << bs_log2) + off) * Dv + (c + x * CP) * E);
      }
    }
    // the U keys of a lane are scored first; the running maximum moves once per batch of U keys, so the accumulators are
    // rescaled once per batch
    float vf[U][VC][E], sc[U][HB];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float kf[E];
      const T* kp_ = reinterpret_cast<const T*>(&kr[u]);
#pragma unroll
      for (int e = 0; e < E; ++e) kf[e] = to_f32<T>(kp_[e]);
#pragma unroll
      for (int x = 0; x < VC; ++x) {
        const T* vp = reinterpret_cast<const T*>(&vr[u][x]);
#pragma unroll
        for (int e = 0; e < E; ++e) vf[u][x][e] = to_f32<T>(vp[e]);
      }
#pragma unroll
      for (int hh = 0; hh < HB; ++hh) {
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < E; ++e) s = fmaf(qv[hh][e], kf[e], s);
        for (int o = CP >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if (capped) s = cap2 * capped_tanh<T>(s);
        sc[u][hh] = valid[u] ? s : -INFINITY;
      }
    }
#pragma unroll
    for (int hh = 0; hh < HB; ++hh) {
      float mn = mx[hh];
#pragma unroll
      for (int u = 0; u < U; ++u) mn = fmaxf(mn, sc[u][hh]);
      const float ms = mn == -INFINITY ? 0.f : mn;       // no key of this lane yet: every term below is 2^(-inf) = 0
      const float r = ex2_approx(mx[hh] - ms);
      mx[hh] = mn;
      l[hh] *= r;
#pragma unroll
      for (int x = 0; x < VC; ++x)
#pragma unroll
        for (int e = 0; e < E; ++e) acc[hh][x][e] *= r;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const float pj = ex2_approx(sc[u][hh] - ms);
        l[hh] += pj;
#pragma unroll
        for (int x = 0; x < VC; ++x)
#pragma unroll
          for (int e = 0; e < E; ++e) acc[hh][x][e] = fmaf(pj, vf[u][x][e], acc[hh][x][e]);
      }
    }
  }
  const int LDW = Dv + 2;
#pragma unroll
  for (int hh = 0; hh < HB; ++hh) {
    for (int o = CP; o < 32; o <<= 1) {
      const float m2 = __shfl_xor_sync(0xffffffffu, mx[hh], o);
      const float l2 = __shfl_xor_sync(0xffffffffu, l[hh], o);
      const float mn = fmaxf(mx[hh], m2);
      const float e1 = mx[hh] == -INFINITY ? 0.f : exp2f(mx[hh] - mn);
      const float e2 = m2 == -INFINITY ? 0.f : exp2f(m2 - mn);
      l[hh] = l[hh] * e1 + l2 * e2;
#pragma unroll
      for (int x = 0; x < VC; ++x)
#pragma unroll
        for (int e = 0; e < E; ++e) {
          const float a2 = __shfl_xor_sync(0xffffffffu, acc[hh][x][e], o);
          acc[hh][x][e] = acc[hh][x][e] * e1 + a2 * e2;
        }
      mx[hh] = mn;
    }
    if (kk == 0) {
      float* w = sm + (warp * HB + hh) * LDW;
      if (c == 0) { w[0] = mx[hh]; w[1] = l[hh]; }
#pragma unroll
      for (int x = 0; x < VC; ++x)
        if (liveV[x]) {
#pragma unroll
          for (int e = 0; e < E; ++e) w[2 + (c + x * CP) * E + e] = acc[hh][x][e];
        }
    }
  }
  __syncthreads();
  const bool direct = M == 1 && nsplit == 1;
  for (int i = threadIdx.x; i < nh * Dv; i += blockDim.x) {
    const int hh = i / Dv, d = i % Dv;
    const int h = h0 + hh;
    float mt = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) mt = fmaxf(mt, sm[(w * HB + hh) * LDW]);
    float lt = 0.f, at = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float* ws = sm + (w * HB + hh) * LDW;
      if (ws[0] != -INFINITY) {
        const float e = exp2f(ws[0] - mt);
        lt += ws[1] * e;
        at += ws[2 + d] * e;
      }
    }
    if (direct) {
      float f = post;
      if (opt.sink) lt += exp2f(opt.sink[h] * kLog2e - mt);
      if (opt.gate) f *= sigmoid_f(opt.gate[(long long)t * opt.ld_gate + h]);
      out[(long long)t * ldo + (long long)h * Dv + d] = from_f32<T>(lt > 0.f ? at / lt * f : 0.f);
    } else {
      float* pr = part + ((((long long)t * H + h) * M + m) * nsplit + split) * LDW;
      if (d == 0) { pr[0] = mt; pr[1] = lt; }
      pr[2 + d] = at;
    }
  }
}

// one warp per (token, head): merges the key ranges of every map, then the combination and the norm
template <typename T>
__global__ void __launch_bounds__(128)
multimap_attn_merge_kernel(const float* __restrict__ part, T* __restrict__ out, long long ldo, int H, long long items, int M, int Dv, int nsplit,
                           int combine, float lambda, float post, float eps, const b200_attn_opts opt) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * 4 + warp;            // (token, head)
  if (item >= items) return;
  const int LDW = Dv + 2;
  float res[kAcc];
#pragma unroll
  for (int a = 0; a < kAcc; ++a) res[a] = 0.f;
  for (int m = 0; m < M; ++m) {
    const float* pr = part + (item * M + m) * nsplit * LDW;
    float mt = -INFINITY;
    for (int s = 0; s < nsplit; ++s) mt = fmaxf(mt, pr[s * LDW]);
    float lt = 0.f, at[kAcc];
#pragma unroll
    for (int a = 0; a < kAcc; ++a) at[a] = 0.f;
    for (int s = 0; s < nsplit; ++s) {
      const float ms = pr[s * LDW];
      if (ms == -INFINITY) continue;
      const float e = exp2f(ms - mt);                    // the recorded maxima are in units of log 2
      lt += pr[s * LDW + 1] * e;
#pragma unroll
      for (int a = 0; a < kAcc; ++a) {
        const int d = lane + 32 * a;
        if (d < Dv) at[a] += pr[s * LDW + 2 + d] * e;
      }
    }
    if (opt.sink) lt += exp2f(opt.sink[item % H] * kLog2e - mt);
    const float inv = lt > 0.f ? 1.f / lt : 0.f;
    const float coef = m == 0 ? 1.f : -lambda;
#pragma unroll
    for (int a = 0; a < kAcc; ++a) res[a] = fmaf(coef, at[a] * inv, res[a]);
  }
  float mult = post;
  if (combine) {
    float ss = 0.f;
#pragma unroll
    for (int a = 0; a < kAcc; ++a) ss += (lane + 32 * a < Dv) ? res[a] * res[a] : 0.f;
    ss = warp_sum(ss);
    mult = rsqrtf(ss / Dv + eps) * post;
  }
  if (opt.gate) mult *= sigmoid_f(opt.gate[item / H * opt.ld_gate + item % H]);
#pragma unroll
  for (int a = 0; a < kAcc; ++a) {
    const int d = lane + 32 * a;
    if (d < Dv) out[item / H * ldo + item % H * Dv + d] = from_f32<T>(res[a] * mult);
  }
}
}  // namespace b200

B200_API int b200_qkv_store(const void* proj, long long ld, const float* bias, const float* wq, const float* wk, const float* cos_t,
                            const float* sin_t, const int* pos, const int* slot, const int* table, int max_blocks, void* q_out,
                            void* ck, void* cv, const void* v_first, const float* v_lambda, int tokens, int H, int G, int M, int D,
                            int Dv, int rot, int block_size, float eps, int has_kv, int x_dtype, int dtype, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || M <= 0 || D <= 0 || rot < 0 || rot > D || (rot & 1) || block_size <= 0 || (has_kv && Dv <= 0)) return B200_ERR_BAD_SHAPE;
  if ((wq && has_kv && !wk) || (v_first && (!v_lambda || !has_kv)) || (rot && (!cos_t || !sin_t))) return B200_ERR_BAD_SHAPE;
  const int big = has_kv && Dv > D ? Dv : D;
  if (big > 512) return B200_ERR_TOO_LARGE;
  const int es = x_dtype == B200_DT_FP32 ? 4 : 2, eo = dtype == B200_DT_FP32 ? 4 : 2;
  auto al = [](const void* p_, int n) { return !(reinterpret_cast<uintptr_t>(p_) & (n - 1)); };
  // two neighbouring pairs per lane: both parts of a row, and where their second halves start, are even
  const bool v2 = D % 4 == 0 && rot % 4 == 0 && (!has_kv || Dv % 4 == 0) && ld % 2 == 0 && al(proj, 2 * es) && al(q_out, 2 * eo) &&
                  (!has_kv || (al(ck, 2 * eo) && al(cv, 2 * eo))) && (!v_first || al(v_first, 2 * eo));
  QkvStoreArgs a;
  a.proj = proj; a.ld = ld; a.bias = bias; a.wq = wq; a.wk = wk; a.cs = cos_t; a.sn = sin_t; a.pos = pos; a.slot = slot; a.table = table;
  a.q_out = q_out; a.ck = ck; a.cv = cv; a.v_first = v_first; a.v_lambda = v_lambda; a.max_blocks = max_blocks; a.tokens = tokens;
  a.QR = H * M; a.KR = G * M; a.G = G; a.D = D; a.Dv = Dv; a.rot = rot; a.block_size = block_size; a.has_kv = has_kv; a.eps = eps;
  a.TB = tokens <= 512 ? 1 : 8;
  const dim3 grid((tokens + a.TB - 1) / a.TB, (a.QR + (has_kv ? a.KR + G : 0) + 3) / 4);
  if (grid.y > 65535) return B200_ERR_TOO_LARGE;
  cudaStream_t st = (cudaStream_t)stream;
#define QS(TX, T, VV, NN) qkv_store_kernel<TX, T, VV, NN><<<grid, 128, 0, st>>>(a)
  // pairs of a row: at most big / 2 + 1
#define QS_V(TX, T)                                                                                                          \
  do {                                                                                                                       \
    if (v2 && big <= 128) QS(TX, T, 2, 1); else if (v2 && big <= 256) QS(TX, T, 2, 2); else if (v2) QS(TX, T, 2, 4);           \
    else if (big <= 62) QS(TX, T, 1, 1); else if (big <= 126) QS(TX, T, 1, 2); else QS(TX, T, 1, 9);                          \
  } while (0)
  if (x_dtype == B200_DT_FP32 && dtype == B200_DT_FP32) QS_V(float, float);
  else if (x_dtype == B200_DT_FP32 && dtype == B200_DT_BF16) QS_V(float, __nv_bfloat16);
  else if (x_dtype == B200_DT_FP32 && dtype == B200_DT_FP16) QS_V(float, __half);
  else if (x_dtype == B200_DT_BF16 && dtype == B200_DT_BF16) QS_V(__nv_bfloat16, __nv_bfloat16);
  else return B200_ERR_UNSUPPORTED;
#undef QS_V
#undef QS
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_qknorm_rope_store(const float* proj, long long ld, const float* wq, const float* wk, const float* cos_t,
                                    const float* sin_t, const int* pos, const int* slot, const int* table, int max_blocks,
                                    void* q_out, void* ck, void* cv, int tokens, int H, int G, int M, int D, int Dv, int rot,
                                    int block_size, float eps, int has_kv, int dtype, void* stream) {
  return b200_qkv_store(proj, ld, nullptr, wq, wk, cos_t, sin_t, pos, slot, table, max_blocks, q_out, ck, cv, nullptr, nullptr, tokens, H,
                        G, M, D, Dv, rot, block_size, eps, has_kv, B200_DT_FP32, dtype, stream);
}

B200_API int b200_conv_qknorm_store(const void* proj, long long ld, const float* bias, const float* w, const float* tail, const int* pos,
                                    const int* slot, const int* table, int max_blocks, void* q_out, void* ck, void* cv, int tokens,
                                    int H, int G, int D, int Dv, int taps, int block_size, float eps, float temp_coef,
                                    float temp_every, int norm_qk, int norm_v, int x_dtype, int dtype, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || D <= 0 || Dv <= 0 || block_size <= 0 || taps < 1 || !(temp_every > 0.f)) return B200_ERR_BAD_SHAPE;
  const int big = D > Dv ? D : Dv;
  if (taps > kConvMaxTaps || big > 512) return B200_ERR_TOO_LARGE;
  const int es = x_dtype == B200_DT_FP32 ? 4 : 2, eo = dtype == B200_DT_FP32 ? 4 : 2;
  auto al = [](const void* p_, int n) { return !(reinterpret_cast<uintptr_t>(p_) & (n - 1)); };
  const bool v2 = D % 2 == 0 && Dv % 2 == 0 && ld % 2 == 0 && al(proj, 2 * es) && al(q_out, 2 * eo) && al(ck, 2 * eo) && al(cv, 2 * eo);
  const int TB = tokens <= 512 ? 1 : 8;
  dim3 grid((tokens + TB - 1) / TB, (H + 2 * G + 3) / 4);
  cudaStream_t st = (cudaStream_t)stream;
#define CQ(TX, T, TAPSV, VV, VIV)                                                                                              \
  conv_qknorm_store_kernel<TX, T, TAPSV, VV, VIV><<<grid, 128, 0, st>>>((const TX*)proj, ld, bias, w, tail, pos, slot, table,   \
      max_blocks, (T*)q_out, (T*)ck, (T*)cv, tokens, H, G, D, Dv, block_size, eps, temp_coef, temp_every, norm_qk, norm_v, TB)
#define CQ_V(TX, T, TAPSV)                                                                                                     \
  do {                                                                                                                         \
    if (v2 && big <= 64) CQ(TX, T, TAPSV, 2, 1); else if (v2 && big <= 128) CQ(TX, T, TAPSV, 2, 2);                             \
    else if (v2 && big <= 256) CQ(TX, T, TAPSV, 2, 4); else if (v2) CQ(TX, T, TAPSV, 2, 8);                                    \
    else if (big <= 128) CQ(TX, T, TAPSV, 1, 4); else CQ(TX, T, TAPSV, 1, 16);                                                 \
  } while (0)
#define CQ_T(TX, T)                                                                                                            \
  switch (taps) {                                                                                                              \
    case 1: CQ_V(TX, T, 1); break; case 2: CQ_V(TX, T, 2); break; case 3: CQ_V(TX, T, 3); break; case 4: CQ_V(TX, T, 4); break; \
    default: CQ_V(TX, T, 5); break;                                                                                            \
  }
  if (x_dtype == B200_DT_BF16 && dtype == B200_DT_BF16) { CQ_T(__nv_bfloat16, __nv_bfloat16) }
  else if (x_dtype == B200_DT_FP32 && dtype == B200_DT_FP32) { CQ_T(float, float) }
  else return B200_ERR_UNSUPPORTED;
#undef CQ_T
#undef CQ_V
#undef CQ
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_multimap_attn_ex(const void* q, const void* ck, const void* cv, const int* pos, const int* slot, const int* table,
                                   int max_blocks, void* out, long long ldo, float* part, int tokens, int H, int G, int M, int D, int Dv,
                                   int block_size, float scale, int window, int keep_first, int nsplit, int combine, float lambda,
                                   float post, float eps, const b200_attn_opts* opts, int dtype, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  const b200_attn_opts opt = opts ? *opts : b200_attn_opts{};
  if (opts && (M != 1 || opt.chunk < 0 || (opt.chunk > 0 && window > 0) || !(opt.softcap >= 0.f))) return B200_ERR_UNSUPPORTED;
  if (H <= 0 || G <= 0 || H % G || M < 1 || M > kMaxMaps || D <= 0 || Dv <= 0 || block_size <= 0 || nsplit < 1) return B200_ERR_BAD_SHAPE;
  if (Dv > kMaxDv) return B200_ERR_TOO_LARGE;
  if (combine && M != 2) return B200_ERR_UNSUPPORTED;
  cudaStream_t st = (cudaStream_t)stream;
  const int rep = H / G;
  {
    // vector kernel: key and value rows of whole 16-byte chunks, at most 32 of them, pages of a power-of-two size
    const int E = dtype == B200_DT_FP32 ? 4 : 8;
    const int CPK = D / E, CPV = Dv / E;
    int bs_log2 = 0;
    while ((1 << bs_log2) < block_size) ++bs_log2;
    if (D % E == 0 && Dv % E == 0 && CPK <= 32 && CPV <= 32 && (1 << bs_log2) == block_size && (part || (M == 1 && nsplit == 1)) &&
        !((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(ck) | reinterpret_cast<uintptr_t>(cv)) & 15)) {
      // lanes per key: the chunks of a key row, or of half a value row if that is more (a lane then holds two value chunks)
      int CP = 1;
      while (CP < CPK || 2 * CP < CPV) CP <<= 1;
      const int VC = CPV > CP ? 2 : 1;
      const int HB = rep >= 4 ? 4 : (rep >= 2 ? 2 : 1);
      const int passes = (rep + HB - 1) / HB;
      const bool direct = M == 1 && nsplit == 1;
      if ((long long)G * passes > 65535 || nsplit * M > 65535) return B200_ERR_TOO_LARGE;
      if (!direct && !part) return B200_ERR_BAD_SHAPE;
      dim3 grid(tokens, G * passes, nsplit * M);
      const size_t smem = (size_t)4 * HB * (Dv + 2) * sizeof(float);
#define MMV2(T, HBV, VCV)                                                                                                    \
  multimap_attn_vec_kernel<T, HBV, VCV><<<grid, 128, smem, st>>>((const T*)q, (const T*)ck, (const T*)cv, pos, slot, table,   \
      max_blocks, (T*)out, ldo, part, H, G, M, D, Dv, bs_log2, scale, window, keep_first, nsplit, post, CP, CPK, CPV, opt)
#define MMV(T, HBV)                                                                                                          \
  do { if (VC == 2) MMV2(T, HBV, 2); else MMV2(T, HBV, 1); } while (0)
#define MMV_T(T)                                                                                                             \
  do {                                                                                                                       \
    if (HB == 4) MMV(T, 4); else if (HB == 2) MMV(T, 2); else MMV(T, 1);                                                     \
    if (!direct)                                                                                                             \
      multimap_attn_merge_kernel<T><<<(unsigned)(((long long)tokens * H + 3) / 4), 128, 0, st>>>(                             \
          part, (T*)out, ldo, H, (long long)tokens * H, M, Dv, nsplit, combine, lambda, post, eps, opt);                             \
  } while (0)
      if (dtype == B200_DT_BF16) MMV_T(__nv_bfloat16);
      else if (dtype == B200_DT_FP16) MMV_T(__half);
      else if (dtype == B200_DT_FP32) MMV_T(float);
      else return B200_ERR_UNSUPPORTED;
#undef MMV_T
#undef MMV
#undef MMV2
      B200_LAUNCH_CHECK();
      return 0;
    }
  }
  const int nw = 4;
  const size_t smem = (size_t)nw * D * 4;
  if (smem > 48 * 1024) return B200_ERR_TOO_LARGE;
  const unsigned grid = (unsigned)(((long long)tokens * H + nw - 1) / nw);
  B200_DISPATCH_T(dtype, multimap_attn_kernel<T><<<grid, nw * 32, smem, st>>>(
      (const T*)q, (const T*)ck, (const T*)cv, pos, slot, table, max_blocks, (T*)out, ldo, tokens, H, G, M, D, Dv, block_size, scale,
      window, keep_first, combine, lambda, post, eps, opt));
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_multimap_attn(const void* q, const void* ck, const void* cv, const int* pos, const int* slot, const int* table,
                                int max_blocks, void* out, long long ldo, float* part, int tokens, int H, int G, int M, int D, int Dv,
                                int block_size, float scale, int window, int keep_first, int nsplit, int combine, float lambda,
                                float post, float eps, int dtype, void* stream) {
  return b200_multimap_attn_ex(q, ck, cv, pos, slot, table, max_blocks, out, ldo, part, tokens, H, G, M, D, Dv, block_size, scale, window,
                               keep_first, nsplit, combine, lambda, post, eps, nullptr, dtype, stream);
}
