// Gated linear attention with a decay per key channel, over the runs of a ragged serving step (see linear_scan.cu for runs,
// state rows and the other scan modes). All arithmetic is fp32.
//
//   b200_lowrank_decay   a[t, c] = sigmoid(sum_r w2[c, r] x[t, r] + bias[c])^(1 / tau), formed as exp(log sigmoid(.) / tau), or
//                        exp(-exp(sum_r w2[c, r] tanh(x[t, r]) + bias[c]))
//   b200_channel_scan    per head, state S [D, Dv] (fp32, in `state` [rows, H, D, Dv]):
//                            S <- diag(g_t) S + k_t v_t^T ;   o_t = S^T q_t                      (u NULL)
//                            o_t = (S + diag(u) k_t v_t^T)^T q_t ;   S <- diag(g_t) S + k_t v_t^T  (u [H, D]: a bonus for the
//                            current token, which the read-out sees before the state decays)
//
// A run is walked token by token, but the recurrence is linear, so a long run need not be walked by one CTA: it is cut into
// tiles (64 tokens), and
//   pass 1  every tile but a run's last forms its local state (from zero) and the product of its decays,
//   carry   per element of S, the tiles of a run are chained: incoming state of tile j + 1 = decay_j * incoming_j + local_j,
//   pass 2  every tile is walked again from its incoming state and writes its outputs; the last one leaves the run's state.
// Runs of at most one tile (decode batches, short pieces) take pass 0: one walk from and to the state row.
//
// Columns of S are independent. A thread owns R rows of CPT columns, LPC lanes share a column and reduce their parts of an
// output by shuffles (each step halves the columns a lane still carries), a CTA owns a block of columns of one (run or tile,
// head). k, q, g and v of a chunk of tokens are staged through shared memory by cp.async, one chunk ahead.
#include "common.cuh"
#include "mma_sync.cuh"
#include "../include/b200_ops.h"

namespace b200 {

constexpr int kCsR = 16, kCsCols = 4;                   // rows and columns of a thread

__device__ __forceinline__ void cs_async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cs_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cs_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cs_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

struct ChannelScanArgs {
  const float *q, *k, *v, *g, *u;
  long long ldq, ldk, ldv, ldg;
  float* state;                                          // [rows, H, D, Dv]
  float* part;                                           // [tiles, H, D, Dv]: local, then incoming states
  float* pdec;                                           // [tiles, H, D]: decay products of the tiles
  const int *runs, *pos, *slot;                          // runs NULL: a decode batch
  const int *tiles, *tile_of;
  float* o;
  int H, G, D, Dv, chunk, vec, vecv;
};

// PASS 0: blockIdx.x is a run; 1, 2: a tile
// Four CTAs per SM for short runs and decode batches (0: the compiler's own choice; the tile passes are faster with it).
template <int PASS, int LPC, bool BONUS>
__global__ void __launch_bounds__(128, PASS == 0 ? 4 : 0)
channel_scan_kernel(const ChannelScanArgs a) {
  extern __shared__ __align__(16) float sm[];
  constexpr int R = kCsR, CPT = kCsCols, RP = R + 4, DP = LPC * RP, cpw = 32 / LPC;
  const int b_ = blockIdx.x, h = blockIdx.y;
  int first, n, p0, s;
  bool from_part = false, keep_state = true;
  if (PASS == 0) {
    if (a.runs) { first = a.runs[4 * b_]; n = a.runs[4 * b_ + 1]; p0 = a.runs[4 * b_ + 2]; s = a.runs[4 * b_ + 3]; }
    else { first = b_; n = 1; p0 = a.pos[b_]; s = a.slot[b_]; }
  } else {
    const int place = a.tile_of[4 * b_ + 1], count = a.tile_of[4 * b_ + 2];
    if (PASS == 1 && place + 1 == count) return;         // nobody asks for the last tile's local state
    first = a.tiles[4 * b_]; n = a.tiles[4 * b_ + 1]; p0 = a.tiles[4 * b_ + 2]; s = a.tiles[4 * b_ + 3];
    from_part = PASS == 2;
    keep_state = PASS == 2 && place + 1 == count;
  }
  const int H = a.H, D = a.D, Dv = a.Dv;
  const int kvh = h / (H / a.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int l = lane % LPC, jj = lane / LPC;             // the lanes of a column are neighbours: an eighth of a warp reads
  const int ncol = nw * cpw * CPT;                       // different rows of a staged token, without bank conflicts
  const int col0 = blockIdx.z * ncol;
  const int cc0 = (warp * cpw + jj) * CPT;               // first column of this thread inside the CTA's block
  const int j0 = col0 + cc0;
  const int row0 = l * R;
  const int CH = a.chunk;
  constexpr int NS = PASS == 1 ? 2 : 3;                  // staged rows per token: k, g and, where there are outputs, q
  const int per = CH * (NS * DP + ncol);                 // floats per buffer
  auto KS = [&](int b) { return sm + b * per; };
  auto GS = [&](int b) { return sm + b * per + CH * DP; };
  auto QS = [&](int b) { return sm + b * per + 2 * CH * DP; };
  auto VS = [&](int b) { return sm + b * per + NS * CH * DP; };
  auto at = [](int d) { return (d / R) * RP + d % R; };  // key channel d -> its place in a staged row
  if (LPC * R > D) {                                     // rows past D never arrive by copy: zero keys keep their state at zero
    const int padw = LPC * R - D;
    for (int i = threadIdx.x; i < 2 * CH * padw; i += blockDim.x) {
      const int b = i / (CH * padw), r = i % (CH * padw);
      const int x = (r / padw) * DP + at(D + r % padw);
      KS(b)[x] = 0.f;
      GS(b)[x] = 0.f;
      if (PASS != 1) QS(b)[x] = 0.f;
    }
  }
  float2 S2[CPT][R / 2];
  float* sp = a.state + ((long long)s * H + h) * D * (long long)Dv;
  float* pp = PASS == 0 ? nullptr : a.part + ((long long)b_ * H + h) * D * (long long)Dv;
  const float* src = from_part ? pp : (PASS == 0 && p0 > 0 ? sp : nullptr);
  const bool v4 = a.vecv && j0 + CPT <= Dv;              // four whole columns on a 16-byte boundary
#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int d = row0 + 2 * i + e;
      float x[CPT];
#pragma unroll
      for (int c = 0; c < CPT; ++c) x[c] = 0.f;
      if (src && d < D) {
        const float* r = src + (long long)d * Dv + j0;
        if (v4) *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(r);
        else {
#pragma unroll
          for (int c = 0; c < CPT; ++c) if (j0 + c < Dv) x[c] = r[c];
        }
      }
#pragma unroll
      for (int c = 0; c < CPT; ++c) { if (e == 0) S2[c][i].x = x[c]; else S2[c][i].y = x[c]; }
    }
  }
  // the first warp of the first column block also multiplies up the decays of its tile
  const bool owns_dec = PASS == 1 && blockIdx.z == 0 && warp == 0;
  float2 P2[R / 2];
#pragma unroll
  for (int i = 0; i < R / 2; ++i) P2[i] = make_float2(1.f, 1.f);

  // the bonus of a thread's rows stays in registers over a tile; a short run reads it per token instead (occupancy)
  float2 u2[R / 2];
  auto load_u = [&]() {
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      u2[i].x = row0 + 2 * i < D ? __ldg(a.u + h * D + row0 + 2 * i) : 0.f;
      u2[i].y = row0 + 2 * i + 1 < D ? __ldg(a.u + h * D + row0 + 2 * i + 1) : 0.f;
    }
  };
  if (BONUS && PASS == 2) load_u();

  auto stage = [&](int b, int c0) {
    const int cn = min(CH, n - c0);
    for (int tt = warp; tt < cn; tt += nw) {
      const long long tr = first + c0 + tt;
      const float* kr = a.k + tr * a.ldk + (long long)kvh * D;
      const float* qr = a.q + tr * a.ldq + (long long)kvh * D;
      const float* gr = a.g + tr * a.ldg + (long long)h * D;
      if (a.vec) {
        for (int d = lane * 4; d < D; d += 128) {
          cs_async16(KS(b) + tt * DP + at(d), kr + d);
          cs_async16(GS(b) + tt * DP + at(d), gr + d);
          if (PASS != 1) cs_async16(QS(b) + tt * DP + at(d), qr + d);
        }
      } else {
        for (int d = lane; d < D; d += 32) {
          cs_async4(KS(b) + tt * DP + at(d), kr + d);
          cs_async4(GS(b) + tt * DP + at(d), gr + d);
          if (PASS != 1) cs_async4(QS(b) + tt * DP + at(d), qr + d);
        }
      }
      const float* vr = a.v + tr * a.ldv + (long long)h * Dv + col0;
      for (int c = lane * 4; c < ncol; c += 128) {
        float* dst = VS(b) + tt * ncol + c;
        if (a.vecv && col0 + c + 4 <= Dv) cs_async16(dst, vr + c);
        else {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            if (col0 + c + e < Dv) cs_async4(dst + e, vr + c + e);
            else dst[e] = 0.f;
          }
        }
      }
    }
  };

  stage(0, 0);
  cs_commit();
  int buf = 0;
  for (int c0 = 0; c0 < n; c0 += CH, buf ^= 1) {
    const int cn = min(CH, n - c0);
    if (c0 + CH < n) stage(buf ^ 1, c0 + CH);
    cs_commit();
    cs_wait<1>();
    __syncthreads();
    const float* ks = KS(buf) + l * RP;
    const float* gs = GS(buf) + l * RP;
    const float* qs = PASS == 1 ? ks : QS(buf) + l * RP;
    const float* vs = VS(buf) + cc0;
    for (int tt = 0; tt < cn; ++tt) {
      float2 k2[R / 2], g2[R / 2], q2[R / 2];
#pragma unroll
      for (int i = 0; i < R / 2; i += 2) {
        const float4 kk = *reinterpret_cast<const float4*>(ks + tt * DP + 2 * i);
        const float4 gg = *reinterpret_cast<const float4*>(gs + tt * DP + 2 * i);
        k2[i] = make_float2(kk.x, kk.y); k2[i + 1] = make_float2(kk.z, kk.w);
        g2[i] = make_float2(gg.x, gg.y); g2[i + 1] = make_float2(gg.z, gg.w);
        if (PASS != 1) {
          const float4 qq = *reinterpret_cast<const float4*>(qs + tt * DP + 2 * i);
          q2[i] = make_float2(qq.x, qq.y); q2[i + 1] = make_float2(qq.z, qq.w);
        }
      }
      const float4 vv = *reinterpret_cast<const float4*>(vs + tt * ncol);
      const float vc[CPT] = {vv.x, vv.y, vv.z, vv.w};
      float o[CPT];
      float bonus = 0.f;                                 // this lane's part of q . diag(u) k, the weight of the token's own value
      if (BONUS && PASS != 1) {
        if (PASS == 0) load_u();
        float2 ba = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < R / 2; ++i) ba = __ffma2_rn(__fmul2_rn(u2[i], k2[i]), q2[i], ba);
        bonus = ba.x + ba.y;
      }
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        const float2 v2 = make_float2(vc[c], vc[c]);
        float2 oa = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
          if (BONUS && PASS != 1) oa = __ffma2_rn(S2[c][i], q2[i], oa);
          S2[c][i] = __ffma2_rn(g2[i], S2[c][i], __fmul2_rn(k2[i], v2));
          if (!BONUS && PASS != 1) oa = __ffma2_rn(S2[c][i], q2[i], oa);
        }
        o[c] = oa.x + oa.y;
        if (BONUS && PASS != 1) o[c] = fmaf(bonus, vc[c], o[c]);
      }
      if (PASS == 1) {
        if (owns_dec) {
#pragma unroll
          for (int i = 0; i < R / 2; ++i) P2[i] = __fmul2_rn(P2[i], g2[i]);
        }
        continue;
      }
      // sum over the LPC lanes of the columns: the first step sends two columns away and keeps two, the second one and one
      float* orow = a.o + ((long long)(first + c0 + tt) * H + h) * Dv;
      if (LPC == 1) {
        if (v4) *reinterpret_cast<float4*>(orow + j0) = make_float4(o[0], o[1], o[2], o[3]);
        else {
#pragma unroll
          for (int c = 0; c < CPT; ++c) if (j0 + c < Dv) orow[j0 + c] = o[c];
        }
      } else {
        const int b0 = l & 1;
        const float s0 = b0 ? o[0] : o[2], s1 = b0 ? o[1] : o[3];
        float r0 = (b0 ? o[2] : o[0]) + __shfl_xor_sync(0xffffffffu, s0, 1);
        float r1 = (b0 ? o[3] : o[1]) + __shfl_xor_sync(0xffffffffu, s1, 1);
        if (LPC == 2) {
          const int j = j0 + 2 * b0;
          if (j < Dv) orow[j] = r0;
          if (j + 1 < Dv) orow[j + 1] = r1;
        } else {
          const int b1 = (l >> 1) & 1;
          float r = (b1 ? r1 : r0) + __shfl_xor_sync(0xffffffffu, b1 ? r0 : r1, 2);
#pragma unroll
          for (int x = 4; x < LPC; x <<= 1) r += __shfl_xor_sync(0xffffffffu, r, x);
          const int j = j0 + 2 * b0 + b1;
          if (l < 4 && j < Dv) orow[j] = r;
        }
      }
    }
    __syncthreads();
  }
  float* dst = PASS == 1 ? pp : (keep_state ? sp : nullptr);
  if (dst) {
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = row0 + 2 * i + e;
        if (d >= D) continue;
        float* r = dst + (long long)d * Dv + j0;
        float x[CPT];
#pragma unroll
        for (int c = 0; c < CPT; ++c) x[c] = e == 0 ? S2[c][i].x : S2[c][i].y;
        if (v4) *reinterpret_cast<float4*>(r) = *reinterpret_cast<const float4*>(x);
        else {
#pragma unroll
          for (int c = 0; c < CPT; ++c) if (j0 + c < Dv) r[c] = x[c];
        }
      }
    }
  }
  if (owns_dec && jj == 0) {
    float* pd = a.pdec + ((long long)b_ * H + h) * D;
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      if (row0 + 2 * i < D) pd[row0 + 2 * i] = P2[i].x;
      if (row0 + 2 * i + 1 < D) pd[row0 + 2 * i + 1] = P2[i].y;
    }
  }
}

// Chains the tiles of every run: part[tile] (local state) becomes the tile's incoming state. A thread owns V neighbouring
// elements of one head's state; the loads do not depend on the chain, so four tiles are in flight.
template <int V>
__global__ void __launch_bounds__(128)
channel_scan_carry_kernel(float* __restrict__ part, const float* __restrict__ pdec, const float* __restrict__ state,
                          const int* __restrict__ runs, const int* __restrict__ run_tiles, int H, int D, int Dv) {
  const int h = blockIdx.y;
  const long long e0 = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (e0 >= (long long)D * Dv) return;
  const int d = (int)(e0 / Dv);                          // V divides Dv: the V elements share a row
  const int t0 = run_tiles[4 * blockIdx.z], count = run_tiles[4 * blockIdx.z + 1];
  const int p0 = runs[4 * blockIdx.z + 2], s = runs[4 * blockIdx.z + 3];
  float S[V];
#pragma unroll
  for (int v = 0; v < V; ++v) S[v] = p0 > 0 ? state[((long long)s * H + h) * D * (long long)Dv + e0 + v] : 0.f;
  const long long ts = (long long)H * D * Dv;
  float* p = part + (long long)t0 * ts + (long long)h * D * Dv + e0;
  const float* g = pdec + ((long long)t0 * H + h) * D + d;
  for (int j0 = 0; j0 < count; j0 += 4) {
    float loc[4][V], dec[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      dec[u] = 0.f;
#pragma unroll
      for (int v = 0; v < V; ++v) loc[u][v] = 0.f;
      if (j0 + u + 1 < count) {                          // the last tile of a run has no local state
        if (V == 4) *reinterpret_cast<float4*>(loc[u]) = *reinterpret_cast<const float4*>(p + (j0 + u) * ts);
        else loc[u][0] = p[(j0 + u) * ts];
        dec[u] = g[(long long)(j0 + u) * H * D];
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (j0 + u < count) {
        if (V == 4) *reinterpret_cast<float4*>(p + (j0 + u) * ts) = *reinterpret_cast<const float4*>(S);
        else p[(j0 + u) * ts] = S[0];
#pragma unroll
        for (int v = 0; v < V; ++v) S[v] = fmaf(dec[u], S[v], loc[u][v]);
      }
    }
  }
}

// CPT channels per thread, kLrTok tokens at a time, `groups` times: x rows of all of them are staged once and broadcast.
// FAST (16-bit models): base-2 hardware exponential and logarithm; their absolute error in log sigmoid, 2e-7, is divided by tau.
// Otherwise a decay near 1 is formed as 1 + expm1(.): it is raised to the power of its whole reach, and expf's small bias would
// add up where the rounding of 1 + expm1 does not.
constexpr int kLrTok = 8;
// CPT channels per thread share the reads of x. RK: the rank at compile time, weights then stay in registers (0: any rank)
// EXPO: the inputs pass tanh as they are staged, and the decay is exp(-exp(z)).
template <bool FAST, int CPT, int RK, bool EXPO>
__global__ void __launch_bounds__(128)
lowrank_decay_kernel(const float* __restrict__ x, long long ldx, const float* __restrict__ w2, const float* __restrict__ bias,
                     float* __restrict__ out, int tokens, int C, int rank, float inv_tau, int groups) {
  extern __shared__ __align__(16) float xall[];          // [groups * kLrTok][rank]
  const int tb = blockIdx.y * kLrTok * groups;
  for (int i = threadIdx.x; i < groups * kLrTok * rank; i += blockDim.x) {
    const int t = i / rank;
    const float xv = tb + t < tokens ? x[(long long)(tb + t) * ldx + i % rank] : 0.f;
    xall[i] = EXPO ? tanhf(xv) : xv;
  }
  __syncthreads();
  const int c0 = blockIdx.x * 128 * CPT + threadIdx.x;   // this thread's channels are 128 apart
  const float* w[CPT];
#pragma unroll
  for (int j = 0; j < CPT; ++j) w[j] = w2 + (long long)min(c0 + 128 * j, C - 1) * rank;
  const bool vec = rank % 4 == 0 && (reinterpret_cast<uintptr_t>(w2) & 15) == 0;
  constexpr int RV = RK / 4 > 0 ? RK / 4 : 1;
  float4 wr[CPT][RV];
  if (RK > 0) {
#pragma unroll
    for (int j = 0; j < CPT; ++j)
#pragma unroll
      for (int i = 0; i < RV; ++i) wr[j][i] = *reinterpret_cast<const float4*>(w[j] + 4 * i);
  }
  for (int gi = 0; gi < groups; ++gi) {
    const int t0 = tb + gi * kLrTok, nt = min(kLrTok, tokens - t0);
    if (nt <= 0) break;
    const float* xs = xall + gi * kLrTok * rank;
    float acc[kLrTok][CPT];
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      const float b = bias[min(c0 + 128 * j, C - 1)];
#pragma unroll
      for (int t = 0; t < kLrTok; ++t) acc[t][j] = b;
    }
    int r = RK;
    if (RK > 0) {
#pragma unroll
      for (int i = 0; i < RV; ++i)
#pragma unroll
        for (int t = 0; t < kLrTok; ++t) {
          const float4 xv = *reinterpret_cast<const float4*>(xs + t * rank + 4 * i);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            acc[t][j] = fmaf(wr[j][i].x, xv.x, acc[t][j]);
            acc[t][j] = fmaf(wr[j][i].y, xv.y, acc[t][j]);
            acc[t][j] = fmaf(wr[j][i].z, xv.z, acc[t][j]);
            acc[t][j] = fmaf(wr[j][i].w, xv.w, acc[t][j]);
          }
        }
    } else if (vec) {
      for (; r < rank; r += 4) {
        float4 wv[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) wv[j] = *reinterpret_cast<const float4*>(w[j] + r);
#pragma unroll
        for (int t = 0; t < kLrTok; ++t) {
          const float4 xv = *reinterpret_cast<const float4*>(xs + t * rank + r);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            acc[t][j] = fmaf(wv[j].x, xv.x, acc[t][j]);
            acc[t][j] = fmaf(wv[j].y, xv.y, acc[t][j]);
            acc[t][j] = fmaf(wv[j].z, xv.z, acc[t][j]);
            acc[t][j] = fmaf(wv[j].w, xv.w, acc[t][j]);
          }
        }
      }
    }
    for (; r < rank; ++r) {
#pragma unroll
      for (int t = 0; t < kLrTok; ++t)
#pragma unroll
        for (int j = 0; j < CPT; ++j) acc[t][j] = fmaf(w[j][r], xs[t * rank + r], acc[t][j]);
    }
#pragma unroll
    for (int t = 0; t < kLrTok; ++t) {
      if (t >= nt) break;
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        const float z = acc[t][j];
        float v;
        if (EXPO) {
          const float y = -expf(z);
          v = FAST ? ex2_approx(y * 1.4426950408889634f) : (y > -0.5f ? 1.f + expm1f(y) : expf(y));
        } else if (FAST) {
          const float z2 = z * 1.4426950408889634f;
          v = ex2_approx((fminf(z2, 0.f) - __log2f(1.f + ex2_approx(-fabsf(z2)))) * inv_tau);
        } else {
          const float y = (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau;        // log sigmoid(z) / tau
          v = y > -0.5f ? 1.f + expm1f(y) : expf(y);
        }
        if (c0 + 128 * j < C) out[(long long)(t0 + t) * C + c0 + 128 * j] = v;
      }
    }
  }
}
}  // namespace b200

// form 0: sigmoid(w2 x + bias)^inv_tau; 1: exp(-exp(w2 tanh(x) + bias))
B200_API int b200_lowrank_decay_ex(const float* x, long long ldx, const float* w2, const float* bias, float* out, int tokens, int C,
                                   int rank, float inv_tau, int form, int fast, void* stream) {
  using namespace b200;
  if (tokens <= 0) return 0;
  if (C <= 0 || rank <= 0 || tokens > 65535 * kLrTok) return B200_ERR_BAD_SHAPE;
  int groups = tokens >= 2048 ? 4 : 1;
  while (groups > 1 && (size_t)groups * kLrTok * rank * 4 > 48 * 1024) groups /= 2;
  const size_t smem = (size_t)groups * kLrTok * rank * 4;
  if (smem > 48 * 1024) return B200_ERR_TOO_LARGE;
  const bool r16 = rank == 16 && !(reinterpret_cast<uintptr_t>(w2) & 15);
  const int cpt = tokens >= 512 ? (r16 ? 2 : 4) : 1;
  dim3 grid((C + 128 * cpt - 1) / (128 * cpt), (tokens + kLrTok * groups - 1) / (kLrTok * groups));
#define LR(FF, CC, RR)                                                                                                         \
  do {                                                                                                                         \
    if (form == 1) lowrank_decay_kernel<FF, CC, RR, true><<<grid, 128, smem, (cudaStream_t)stream>>>(x, ldx, w2, bias, out, tokens, C, rank, inv_tau, groups); \
    else lowrank_decay_kernel<FF, CC, RR, false><<<grid, 128, smem, (cudaStream_t)stream>>>(x, ldx, w2, bias, out, tokens, C, rank, inv_tau, groups); \
  } while (0)
#define LR_F(FF)                                                                                                               \
  do { if (cpt == 2) LR(FF, 2, 16); else if (cpt == 4) LR(FF, 4, 0); else if (r16) LR(FF, 1, 16); else LR(FF, 1, 0); } while (0)
  if (fast) LR_F(true); else LR_F(false);
#undef LR_F
#undef LR
  B200_LAUNCH_CHECK();
  return 0;
}

B200_API int b200_lowrank_decay(const float* x, long long ldx, const float* w2, const float* bias, float* out, int tokens, int C,
                                int rank, float inv_tau, int fast, void* stream) {
  return b200_lowrank_decay_ex(x, ldx, w2, bias, out, tokens, C, rank, inv_tau, 0, fast, stream);
}

B200_API int b200_channel_scan(const float* q, long long ldq, const float* k, long long ldk, const float* v, long long ldv,
                               const float* g, long long ldg, const float* u, float* state, float* part, float* pdec, const int* runs, int n_runs,
                               const int* tiles, int n_tiles, const int* tile_of, const int* run_tiles, int chunk, const int* pos, const int* slot, float* o,
                               int H, int G, int D, int Dv, void* stream) {
  using namespace b200;
  if (n_runs <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || Dv <= 0 || H > 65535 || chunk < 1) return B200_ERR_BAD_SHAPE;
  if (n_tiles > 0 && (!part || !pdec || !tiles || !tile_of || !run_tiles || !runs || n_runs > 65535)) return B200_ERR_BAD_SHAPE;
  int LPC = 1;
  while (LPC * kCsR < D) LPC *= 2;
  if (LPC > 32) return B200_ERR_TOO_LARGE;
  const int wcol = 32 / LPC * kCsCols;                   // columns of a warp
  int nw = 4;
  while (nw > 1 && (nw - 1) * wcol >= Dv) --nw;          // no warp without columns
  const int ncol = nw * wcol, zb = (Dv + ncol - 1) / ncol;
  const int DP = LPC * (kCsR + 4);
  int CH = chunk < 16 ? chunk : 16;
  auto bytes = [&](int ch) { return (size_t)2 * ch * (3 * DP + ncol) * 4; };
  while (CH > 1 && bytes(CH) > 100 * 1024) CH /= 2;
  auto al = [](const void* p_, long long ld) { return !(reinterpret_cast<uintptr_t>(p_) & 15) && ld % 4 == 0; };
  ChannelScanArgs a;
  a.q = q; a.k = k; a.v = v; a.g = g; a.u = u; a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.ldg = ldg;
  a.state = state; a.part = part; a.pdec = pdec; a.runs = runs; a.pos = pos; a.slot = slot; a.tiles = tiles; a.tile_of = tile_of;
  a.o = o; a.H = H; a.G = G; a.D = D; a.Dv = Dv; a.chunk = CH;
  a.vec = D % 4 == 0 && al(q, ldq) && al(k, ldk) && al(g, ldg);
  a.vecv = Dv % 4 == 0 && al(v, ldv) && al(state, 4) && al(o, 4) && (!part || al(part, 4));
  cudaStream_t st = (cudaStream_t)stream;
  const size_t smem = bytes(CH);
#define CS(PASS, LL, NB) do { if (u) CS_B(PASS, LL, NB, true); else CS_B(PASS, LL, NB, false); } while (0)
#define CS_B(PASS, LL, NB, BB)                                                                                             \
  do {                                                                                                                     \
    auto kern = channel_scan_kernel<PASS, LL, (PASS != 1 && BB)>;                                                                             \
    if (smem > 48 * 1024) B200_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));  \
    kern<<<dim3(NB, H, zb), nw * 32, smem, st>>>(a);                                                                       \
  } while (0)
#define CS_L(PASS, NB)                                                                                                     \
  do {                                                                                                                     \
    if (LPC == 1) CS(PASS, 1, NB); else if (LPC == 2) CS(PASS, 2, NB); else if (LPC == 4) CS(PASS, 4, NB);                  \
    else if (LPC == 8) CS(PASS, 8, NB); else if (LPC == 16) CS(PASS, 16, NB); else CS(PASS, 32, NB);                        \
  } while (0)
  if (n_tiles <= 0) {
    CS_L(0, n_runs);
  } else {
    CS_L(1, n_tiles);
    const int V = Dv % 4 == 0 && al(part, 4) ? 4 : 1;
    const long long n = (long long)D * Dv / V;
    dim3 grid((unsigned)((n + 127) / 128), H, n_runs);
    if (V == 4) channel_scan_carry_kernel<4><<<grid, 128, 0, st>>>(part, pdec, state, runs, run_tiles, H, D, Dv);
    else channel_scan_carry_kernel<1><<<grid, 128, 0, st>>>(part, pdec, state, runs, run_tiles, H, D, Dv);
    CS_L(2, n_tiles);
  }
#undef CS_L
#undef CS_B
#undef CS
  B200_LAUNCH_CHECK();
  return 0;
}
