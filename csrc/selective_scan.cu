// Selective state space with a decay per channel and state, over the runs of a ragged serving step (see linear_scan.cu for
// runs and state rows). Per sequence the state S [N, I] (fp32; channels are neighbours in memory) follows
//
//   s_c = softplus(dt_c + bias_c) ;  S[n, c] <- exp(s_c A[n, c]) S[n, c] + s_c u_c B_n
//   y_c = (sum_n S[n, c] C_n + D_c u_c) silu(gate_c) scale
//
// A thread owns one channel and R states of it; LPC lanes share a channel when there are more than 16 states and add their
// parts of y by shuffles. B and C of a chunk of tokens sit in shared memory in fp32 and are read as broadcast 16-byte rows;
// dt, u and the gate are read channel by channel, coalesced, four tokens ahead.
//
// Runs longer than a tile (64 tokens) are cut into tiles, like the channel scan: pass 1 forms every tile's local state and the
// sum of its step sizes (the decay of a tile is exp(A sum s)), the carry chains the tiles of a run, pass 2 walks every
// tile from its incoming state and writes y. Shorter runs and decode batches take pass 0, one walk.
//
// The decays take one exponential per state, channel and token, which is the kernel's cost: 16-bit runs form them in base 2 on
// the special-function unit (A is scaled by log2 e once per thread), fp32 runs as 1 + expm1f(.), whose rounding has no bias
// that a long memory would add up.
#include "common.cuh"
#include "mma_sync.cuh"
#include "../include/b200_ops.h"

namespace b200 {

struct SelScanArgs {
  const void *u, *B, *C, *gate;
  const float *dt, *dt_bias, *A, *D;
  long long ldu, lddt, ldB, ldC, ldg, ldy;
  float* state;                                          // [rows, N, I]
  float* part;                                           // [tiles, N, I] local, then incoming states; then [tiles, I] step sums
  void* y;
  float scale;
  const int *runs, *pos, *slot, *tiles, *tile_of, *run_tiles;
  int n_tiles, inner, N, chunk;
};

__device__ __forceinline__ float decay_exact(float x) { return x > -0.5f ? 1.f + expm1f(x) : expf(x); }

// PASS 0: blockIdx.x is a run, 3: a token (a decode batch); 1, 2: a tile
template <typename T, int R, int LPC, int PASS>
__global__ void __launch_bounds__(128)
selective_scan_kernel(const SelScanArgs a) {
  extern __shared__ __align__(16) float sm[];            // [chunk][B: NP | C: NP]
  constexpr bool exact = sizeof(T) == 4;
  constexpr int NP = R * LPC, cpw = 32 / LPC, U = PASS == 3 ? 1 : 4;
  const int b_ = blockIdx.x;
  int first, n, p0, s;
  bool last_tile = true;
  if (PASS == 0) { first = a.runs[4 * b_]; n = a.runs[4 * b_ + 1]; p0 = a.runs[4 * b_ + 2]; s = a.runs[4 * b_ + 3]; }
  else if (PASS == 3) { first = b_; n = 1; p0 = a.pos[b_]; s = a.slot[b_]; }
  else {
    last_tile = a.tile_of[4 * b_ + 1] + 1 == a.tile_of[4 * b_ + 2];
    if (PASS == 1 && last_tile) return;
    first = a.tiles[4 * b_]; n = a.tiles[4 * b_ + 1]; p0 = a.tiles[4 * b_ + 2]; s = a.tiles[4 * b_ + 3];
  }
  const int inner = a.inner, N = a.N;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int l = lane / cpw, jj = lane % cpw;             // neighbouring lanes own neighbouring channels
  const int c = blockIdx.y * (4 * cpw) + warp * cpw + jj;
  const bool live = c < inner;
  const int cl = live ? c : inner - 1;                   // idle lanes repeat the last channel's loads and store nothing
  const int n0 = l * R;
  float2 S2[R / 2], A2[R / 2];
  float* sp = a.state + (long long)s * N * inner + cl;
  float* pp = PASS == 0 || PASS == 3 ? nullptr : a.part + (long long)b_ * N * inner + cl;
  const float* src = PASS == 2 ? pp : (PASS != 1 && p0 > 0 ? sp : nullptr);
#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
    float av[2], sv[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int st = n0 + 2 * i + e;
      av[e] = st < N ? a.A[(long long)st * inner + cl] * (exact ? 1.f : 1.4426950408889634f) : 0.f;
      sv[e] = src && st < N ? src[(long long)st * inner] : 0.f;
    }
    A2[i] = make_float2(av[0], av[1]);
    S2[i] = make_float2(sv[0], sv[1]);
  }
  const float bias = a.dt_bias[cl], Dc = PASS == 1 ? 0.f : a.D[cl];
  const T* u = reinterpret_cast<const T*>(a.u) + (long long)first * a.ldu + cl;
  const float* dt = a.dt + (long long)first * a.lddt + cl;
  const T* gate = a.gate ? reinterpret_cast<const T*>(a.gate) + (long long)first * a.ldg + cl : nullptr;
  T* y = reinterpret_cast<T*>(a.y) + (long long)first * a.ldy + cl;
  float dsum = 0.f;

  for (int c0 = 0; c0 < n; c0 += a.chunk) {
    const int cn = min(a.chunk, n - c0);
    __syncthreads();
    for (int i = threadIdx.x; i < cn * 2 * NP; i += blockDim.x) {
      const int t = i / (2 * NP), x = i % (2 * NP);
      const int st = x < NP ? x : x - NP;
      float v = 0.f;
      if (st < N && (PASS != 1 || x < NP))
        v = x < NP ? to_f32<T>(reinterpret_cast<const T*>(a.B)[(long long)(first + c0 + t) * a.ldB + st])
                   : to_f32<T>(reinterpret_cast<const T*>(a.C)[(long long)(first + c0 + t) * a.ldC + st]);
      sm[i] = v;
    }
    __syncthreads();
    float du_n[U], dd_n[U], dg_n[U];
    auto fetch = [&](int t) {
#pragma unroll
      for (int x = 0; x < U; ++x) {
        const int tt = min(t + x, cn - 1);
        du_n[x] = to_f32<T>(u[(long long)(c0 + tt) * a.ldu]);
        dd_n[x] = dt[(long long)(c0 + tt) * a.lddt];
        dg_n[x] = (PASS != 1 && gate) ? to_f32<T>(gate[(long long)(c0 + tt) * a.ldg]) : 0.f;
      }
    };
    fetch(0);
    for (int t0 = 0; t0 < cn; t0 += U) {
      float uv[U], dv[U], gv[U];
#pragma unroll
      for (int x = 0; x < U; ++x) { uv[x] = du_n[x]; dv[x] = dd_n[x]; gv[x] = dg_n[x]; }
      if (t0 + U < cn) fetch(t0 + U);
#pragma unroll
      for (int x = 0; x < U; ++x) {
        const int tt = t0 + x;
        if (tt >= cn) break;
        const float z = dv[x] + bias;
        const float sv = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));      // softplus without a threshold
        if (PASS == 1) dsum += sv;
        const float du = sv * uv[x];
        const float2 s2 = make_float2(sv, sv), du2 = make_float2(du, du);
        const float* bs = sm + tt * 2 * NP + n0;
        const float* cs = bs + NP;
        float2 ya = make_float2(0.f, 0.f), yb = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < R / 2; i += 2) {
          const float4 b4 = *reinterpret_cast<const float4*>(bs + 2 * i);
          float2 xa = __fmul2_rn(A2[i], s2), xb = __fmul2_rn(A2[i + 1], s2);
          if (exact) {
            xa = make_float2(decay_exact(xa.x), decay_exact(xa.y));
            xb = make_float2(decay_exact(xb.x), decay_exact(xb.y));
          } else {
            xa = make_float2(ex2_approx(xa.x), ex2_approx(xa.y));
            xb = make_float2(ex2_approx(xb.x), ex2_approx(xb.y));
          }
          S2[i] = __ffma2_rn(xa, S2[i], __fmul2_rn(make_float2(b4.x, b4.y), du2));
          S2[i + 1] = __ffma2_rn(xb, S2[i + 1], __fmul2_rn(make_float2(b4.z, b4.w), du2));
          if (PASS != 1) {
            const float4 c4 = *reinterpret_cast<const float4*>(cs + 2 * i);
            ya = __ffma2_rn(S2[i], make_float2(c4.x, c4.y), ya);
            yb = __ffma2_rn(S2[i + 1], make_float2(c4.z, c4.w), yb);
          }
        }
        if (PASS == 1) continue;
        float yv = (ya.x + ya.y) + (yb.x + yb.y);
#pragma unroll
        for (int o = cpw; o < 32; o <<= 1) yv += __shfl_xor_sync(0xffffffffu, yv, o);
        yv = fmaf(Dc, uv[x], yv);
        if (gate) yv *= gv[x] / (1.f + (exact ? expf(-gv[x]) : __expf(-gv[x])));
        if (l == 0 && live) y[(long long)(c0 + tt) * a.ldy] = from_f32<T>(yv * a.scale);
      }
    }
  }
  float* dst = PASS == 1 ? pp : (last_tile ? sp : nullptr);
  if (dst && live) {
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      if (n0 + 2 * i < N) dst[(long long)(n0 + 2 * i) * inner] = S2[i].x;
      if (n0 + 2 * i + 1 < N) dst[(long long)(n0 + 2 * i + 1) * inner] = S2[i].y;
    }
  }
  if (PASS == 1 && l == 0 && live) a.part[(long long)a.n_tiles * N * inner + (long long)b_ * inner + c] = dsum;
}

// one thread per (state, channel) of a run: chains the run's tiles
__global__ void __launch_bounds__(128)
selective_scan_carry_kernel(float* __restrict__ part, const float* __restrict__ A, const float* __restrict__ state,
                            const int* __restrict__ runs, const int* __restrict__ run_tiles, int n_tiles, int inner, int N) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, st = blockIdx.y;
  if (c >= inner) return;
  const int t0 = run_tiles[4 * blockIdx.z], count = run_tiles[4 * blockIdx.z + 1];
  const int p0 = runs[4 * blockIdx.z + 2], s = runs[4 * blockIdx.z + 3];
  const float a = A[(long long)st * inner + c];
  float S = p0 > 0 ? state[((long long)s * N + st) * inner + c] : 0.f;
  const long long ts = (long long)N * inner;
  float* p = part + (long long)t0 * ts + (long long)st * inner + c;
  const float* ds = part + (long long)n_tiles * ts + (long long)t0 * inner + c;
  for (int j0 = 0; j0 < count; j0 += 4) {
    float loc[4], dec[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const bool has = j0 + u + 1 < count;               // the last tile of a run has no local state
      loc[u] = has ? p[(j0 + u) * ts] : 0.f;
      dec[u] = has ? ds[(long long)(j0 + u) * inner] : 0.f;
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (j0 + u < count) {
        p[(j0 + u) * ts] = S;
        S = fmaf(expf(a * dec[u]), S, loc[u]);
      }
    }
  }
}

template <typename T, int R, int LPC>
static int sel_launch(const SelScanArgs& a, int n_runs, cudaStream_t st) {
  constexpr int NP = R * LPC, CB = 4 * (32 / LPC);
  const unsigned cb = (unsigned)((a.inner + CB - 1) / CB);
  const size_t smem = (size_t)a.chunk * 2 * NP * 4;
#define SEL(PASS, NB)                                                                                                      \
  do {                                                                                                                     \
    auto kern = selective_scan_kernel<T, R, LPC, PASS>;                                                                    \
    if (smem > 48 * 1024) B200_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));  \
    kern<<<dim3(NB, cb), 128, smem, st>>>(a);                                                                              \
  } while (0)
  if (!a.runs) {
    SEL(3, n_runs);
  } else if (a.n_tiles <= 0) {
    SEL(0, n_runs);
  } else {
    SEL(1, a.n_tiles);
    selective_scan_carry_kernel<<<dim3((a.inner + 127) / 128, a.N, n_runs), 128, 0, st>>>(a.part, a.A, a.state, a.runs, a.run_tiles,
                                                                                          a.n_tiles, a.inner, a.N);
    SEL(2, a.n_tiles);
  }
#undef SEL
  B200_LAUNCH_CHECK();
  return 0;
}

template <typename T>
static int sel_dispatch(const SelScanArgs& a, int n_runs, cudaStream_t st) {
  if (a.N <= 4) return sel_launch<T, 4, 1>(a, n_runs, st);
  if (a.N <= 8) return sel_launch<T, 8, 1>(a, n_runs, st);
  if (a.N <= 16) return sel_launch<T, 16, 1>(a, n_runs, st);
  if (a.N <= 32) return sel_launch<T, 16, 2>(a, n_runs, st);
  if (a.N <= 64) return sel_launch<T, 16, 4>(a, n_runs, st);
  if (a.N <= 128) return sel_launch<T, 16, 8>(a, n_runs, st);
  if (a.N <= 256) return sel_launch<T, 16, 16>(a, n_runs, st);
  return B200_ERR_TOO_LARGE;
}
}  // namespace b200

B200_API int b200_selective_scan(const void* u, long long ldu, const float* dt, long long lddt, const float* dt_bias, const void* B,
                                 long long ldB, const void* C, long long ldC, const float* A, const float* D, float* state,
                                 float* part, const void* gate, long long ldg, float scale, void* y, long long ldy, const int* runs,
                                 int n_runs, const int* tiles, int n_tiles, const int* tile_of, const int* run_tiles, const int* pos, const int* slot,
                                 int inner, int N, int dtype, void* stream) {
  using namespace b200;
  if (n_runs <= 0) return 0;
  if (inner <= 0 || N <= 0) return B200_ERR_BAD_SHAPE;
  if (n_tiles > 0 && (!part || !tiles || !tile_of || !run_tiles || !runs || n_runs > 65535)) return B200_ERR_BAD_SHAPE;
  SelScanArgs a;
  a.u = u; a.B = B; a.C = C; a.gate = gate; a.dt = dt; a.dt_bias = dt_bias; a.A = A; a.D = D;
  a.ldu = ldu; a.lddt = lddt; a.ldB = ldB; a.ldC = ldC; a.ldg = ldg; a.ldy = ldy;
  a.state = state; a.part = part; a.y = y; a.scale = scale; a.runs = runs; a.pos = pos; a.slot = slot; a.tiles = tiles;
  a.tile_of = tile_of; a.run_tiles = run_tiles; a.n_tiles = n_tiles; a.inner = inner; a.N = N;
  a.chunk = !runs ? 1 : (N <= 64 ? 64 : 16);
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == B200_DT_BF16) return sel_dispatch<__nv_bfloat16>(a, n_runs, st);
  if (dtype == B200_DT_FP32) return sel_dispatch<float>(a, n_runs, st);
  return B200_ERR_UNSUPPORTED;
}
