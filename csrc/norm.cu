// K5 — RMSNorm / LayerNorm forward and backward, with the residual add fused in.
//
// One CTA per row; 128-bit loads; statistics in fp32. The forward optionally adds a residual
// stream first and writes the sum back (h = x + res; y = norm(h)), so a transformer block touches
// the hidden state once per norm instead of three times. The backward produces dx (plus the
// gradient flowing into the residual stream) and per-CTA partial dw/db rows in a caller-provided
// scratch buffer that a second kernel reduces — no atomics, bitwise reproducible.
//
// Replaces the ATen kernels behind nn.LayerNorm in GPTLike
// (LLM_Distributed_Trainning/PyTorch/ddp_basics/ddp_gpt_wikitext2.py:99-116) and behind HF
// Qwen3RMSNorm in every Fine-Tuning/*.py script (fp32 statistics, eps 1e-6, weight scale).
#include "common.cuh"
#include "../include/b200_ops.h"

namespace b200 {

constexpr int kNormThreads = 256;

template <typename T> struct Vec8 { static constexpr int N = 16 / sizeof(T); };

template <typename T, int N>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[N]) {
  uint4 raw = *reinterpret_cast<const uint4*>(p);
  const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = to_f32<T>(e[i]);
}
template <typename T, int N>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[N]) {
  uint4 raw;
  T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
  for (int i = 0; i < N; ++i) e[i] = from_f32<T>(v[i]);
  *reinterpret_cast<uint4*>(p) = raw;
}

// ---------------------------------------------------------------------------------------------
// forward:  h = x (+ res);  y = (h - mean) * rstd * w (+ b)      [mean = 0 for RMSNorm]
// x, res, y, h_out: [rows, cols] of T;  w, b: [cols] of WT;  stats: [rows, 2] fp32 (mean, rstd)
// ---------------------------------------------------------------------------------------------
template <typename T, typename WT, bool kLayerNorm>
__global__ void __launch_bounds__(kNormThreads)
norm_fwd_kernel(const T* __restrict__ x, const T* __restrict__ res, const WT* __restrict__ w,
                const WT* __restrict__ b, T* __restrict__ y, T* __restrict__ h_out,
                float* __restrict__ stats, int cols, float eps) {
  constexpr int V = 16 / sizeof(T);
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  const T* xr = x + row * cols;
  const T* rr = res ? res + row * cols : nullptr;
  T* yr = y + row * cols;
  T* hr = h_out ? h_out + row * cols : nullptr;
  const int nvec = cols / V;

  float s1 = 0.f, s2 = 0.f;
  for (int i = threadIdx.x; i < nvec; i += blockDim.x) {
    float v[V];
    load_vec<T, V>(xr + i * V, v);
    if (rr) {
      float r[V];
      load_vec<T, V>(rr + i * V, r);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] += r[j];
      if (hr) {
        // round the sum to T first so forward and backward see the same hidden state
        store_vec<T, V>(hr + i * V, v);
      }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) {
      float t = to_f32<T>(from_f32<T>(v[j]));
      s1 += t;
      s2 += t * t;
    }
  }
  s1 = block_sum(s1, red);
  s2 = block_sum(s2, red);
  float mean = 0.f, var;
  if (kLayerNorm) {
    mean = s1 / cols;
    var = fmaxf(s2 / cols - mean * mean, 0.f);
  } else {
    var = s2 / cols;
  }
  const float rstd = rsqrtf(var + eps);
  if (threadIdx.x == 0 && stats) {
    stats[row * 2] = mean;
    stats[row * 2 + 1] = rstd;
  }
  const T* src = (rr && hr) ? hr : xr;  // re-read (L1/L2 hit) instead of keeping the row in registers
  for (int i = threadIdx.x; i < nvec; i += blockDim.x) {
    float v[V];
    load_vec<T, V>(src + i * V, v);
    if (rr && !hr) {
      float r[V];
      load_vec<T, V>(rr + i * V, r);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = to_f32<T>(from_f32<T>(v[j] + r[j]));
    }
    float o[V];
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const int c = i * V + j;
      float t = (v[j] - mean) * rstd * to_f32<WT>(w[c]);
      if (b) t += to_f32<WT>(b[c]);
      o[j] = t;
    }
    store_vec<T, V>(yr + i * V, o);
  }
}

// ---------------------------------------------------------------------------------------------
// backward. Each CTA walks rows blockIdx.x, +gridDim.x, ... and keeps its dw/db partial sums in
// registers (thread t owns column vectors t, t+blockDim, ...), so the partials need one store
// per CTA. dx = rstd * (g - mean(g) - xhat * mean(g * xhat)) with g = dy * w (RMSNorm drops the
// mean(g) term). dres_in (optional) is added to dx: the gradient arriving on the residual path.
// ---------------------------------------------------------------------------------------------
template <typename T, typename WT, bool kLayerNorm, int kMaxVecPerThread>
__global__ void __launch_bounds__(kNormThreads)
norm_bwd_kernel(const T* __restrict__ dy, const T* __restrict__ h, const WT* __restrict__ w,
                const float* __restrict__ stats, const T* __restrict__ dres_in, T* __restrict__ dx,
                float* __restrict__ dw_part, float* __restrict__ db_part, int rows, int cols) {
  constexpr int V = 16 / sizeof(T);
  __shared__ float red[32];
  const int nvec = cols / V;
  float dw_acc[kMaxVecPerThread][V];
  float db_acc[kMaxVecPerThread][V];
#pragma unroll
  for (int k = 0; k < kMaxVecPerThread; ++k)
#pragma unroll
    for (int j = 0; j < V; ++j) dw_acc[k][j] = db_acc[k][j] = 0.f;

  for (long long row = blockIdx.x; row < rows; row += gridDim.x) {
    const T* dyr = dy + row * cols;
    const T* hr = h + row * cols;
    const float mean = stats[row * 2], rstd = stats[row * 2 + 1];
    float sg = 0.f, sgx = 0.f;
#pragma unroll
    for (int k = 0; k < kMaxVecPerThread; ++k) {
      const int i = threadIdx.x + k * kNormThreads;
      if (i < nvec) {
        float g[V], xv[V];
        load_vec<T, V>(dyr + i * V, g);
        load_vec<T, V>(hr + i * V, xv);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          const float xh = (xv[j] - mean) * rstd;
          const float gw = g[j] * to_f32<WT>(w[i * V + j]);
          sg += gw;
          sgx += gw * xh;
          if (dw_part) dw_acc[k][j] += g[j] * xh;
          if (db_part) db_acc[k][j] += g[j];
        }
      }
    }
    sg = block_sum(sg, red);
    sgx = block_sum(sgx, red);
    const float mg = kLayerNorm ? sg / cols : 0.f;
    const float mgx = sgx / cols;
#pragma unroll
    for (int k = 0; k < kMaxVecPerThread; ++k) {
      const int i = threadIdx.x + k * kNormThreads;
      if (i < nvec) {
        float g[V], xv[V], o[V];
        load_vec<T, V>(dyr + i * V, g);
        load_vec<T, V>(hr + i * V, xv);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          const float xh = (xv[j] - mean) * rstd;
          const float gw = g[j] * to_f32<WT>(w[i * V + j]);
          o[j] = rstd * (gw - mg - xh * mgx);
        }
        if (dres_in) {
          float r[V];
          load_vec<T, V>(dres_in + row * cols + i * V, r);
#pragma unroll
          for (int j = 0; j < V; ++j) o[j] += r[j];
        }
        store_vec<T, V>(dx + row * cols + i * V, o);
      }
    }
  }
  if (dw_part || db_part) {
#pragma unroll
    for (int k = 0; k < kMaxVecPerThread; ++k) {
      const int i = threadIdx.x + k * kNormThreads;
      if (i < nvec) {
#pragma unroll
        for (int j = 0; j < V; ++j) {
          if (dw_part) dw_part[(long long)blockIdx.x * cols + i * V + j] = dw_acc[k][j];
          if (db_part) db_part[(long long)blockIdx.x * cols + i * V + j] = db_acc[k][j];
        }
      }
    }
  }
}

// sum the per-CTA partial rows: out[c] (+)= sum_p part[p, c]
template <typename WT>
__global__ void reduce_partials_kernel(const float* __restrict__ part, WT* __restrict__ out, int nparts, int cols,
                                       int accumulate) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= cols) return;
  float s = 0.f;
  for (int p = 0; p < nparts; ++p) s += part[(long long)p * cols + c];
  if (accumulate) s += to_f32<WT>(out[c]);
  out[c] = from_f32<WT>(s);
}

template <typename T, typename WT>
static int launch_norm_fwd(int layer_norm, const void* x, const void* res, const void* w, const void* b, void* y,
                           void* h_out, float* stats, int rows, int cols, float eps, cudaStream_t st) {
  if (layer_norm)
    return (int)launch_pdl(norm_fwd_kernel<T, WT, true>, rows, kNormThreads, 0, st, (const T*)x, (const T*)res, (const WT*)w,
                           (const WT*)b, (T*)y, (T*)h_out, stats, cols, eps);
  return (int)launch_pdl(norm_fwd_kernel<T, WT, false>, rows, kNormThreads, 0, st, (const T*)x, (const T*)res, (const WT*)w,
                         (const WT*)b, (T*)y, (T*)h_out, stats, cols, eps);
}

template <typename T, typename WT, int MV>
static int launch_norm_bwd(int layer_norm, const void* dy, const void* h, const void* w, const float* stats,
                           const void* dres, void* dx, float* dwp, float* dbp, int rows, int cols, int grid,
                           cudaStream_t st) {
  if (layer_norm)
    norm_bwd_kernel<T, WT, true, MV><<<grid, kNormThreads, 0, st>>>((const T*)dy, (const T*)h, (const WT*)w, stats,
                                                                   (const T*)dres, (T*)dx, dwp, dbp, rows, cols);
  else
    norm_bwd_kernel<T, WT, false, MV><<<grid, kNormThreads, 0, st>>>((const T*)dy, (const T*)h, (const WT*)w, stats,
                                                                    (const T*)dres, (T*)dx, dwp, dbp, rows, cols);
  B200_LAUNCH_CHECK();
  return 0;
}

}  // namespace b200
using namespace b200;

// dtype: activations; wdtype: weight/bias/grad-of-weight dtype. cols must be a multiple of 8 (bf16/fp16)
// or 4 (fp32) and at most 8192 * (4 / sizeof(T)) ... see the checks below.
B200_API int b200_norm_fwd(int layer_norm, const void* x, const void* res, const void* w, const void* b, void* y,
                           void* h_out, float* stats, int rows, int cols, float eps, int dtype, int wdtype,
                           void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  const int V = dtype == B200_DT_FP32 ? 4 : 8;
  if (rows <= 0 || cols <= 0 || cols % V) return B200_ERR_BAD_SHAPE;
  if (dtype == B200_DT_BF16 && wdtype == B200_DT_BF16)
    return launch_norm_fwd<__nv_bfloat16, __nv_bfloat16>(layer_norm, x, res, w, b, y, h_out, stats, rows, cols, eps, st);
  if (dtype == B200_DT_BF16 && wdtype == B200_DT_FP32)
    return launch_norm_fwd<__nv_bfloat16, float>(layer_norm, x, res, w, b, y, h_out, stats, rows, cols, eps, st);
  if (dtype == B200_DT_FP32 && wdtype == B200_DT_FP32)
    return launch_norm_fwd<float, float>(layer_norm, x, res, w, b, y, h_out, stats, rows, cols, eps, st);
  if (dtype == B200_DT_FP16 && wdtype == B200_DT_FP16)
    return launch_norm_fwd<__half, __half>(layer_norm, x, res, w, b, y, h_out, stats, rows, cols, eps, st);
  return B200_ERR_UNSUPPORTED;
}

// Number of CTAs (= partial rows) the backward uses for `rows` rows; scratch must hold
// 2 * b200_norm_bwd_parts(rows) * cols floats when dw/db are requested.
B200_API int b200_norm_bwd_parts(int rows) {
  int g = 2 * kNumSMs;
  return rows < g ? rows : g;
}

B200_API int b200_norm_bwd(int layer_norm, const void* dy, const void* h, const void* w, const float* stats,
                           const void* dres_in, void* dx, void* dw, void* db, float* scratch, int accumulate,
                           int rows, int cols, int dtype, int wdtype, void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  const int V = dtype == B200_DT_FP32 ? 4 : 8;
  if (rows <= 0 || cols <= 0 || cols % V) return B200_ERR_BAD_SHAPE;
  const int nvec = cols / V;
  const int mv = ceil_div(nvec, kNormThreads);
  if (mv > 4) return B200_ERR_TOO_LARGE;  // cols <= 8192 (16-bit) / 4096 (fp32)
  if ((dw || db) && !scratch) return B200_ERR_BAD_SHAPE;
  const int grid = b200_norm_bwd_parts(rows);
  float* dwp = dw ? scratch : nullptr;
  float* dbp = db ? scratch + (long long)grid * cols : nullptr;
  int rc = B200_ERR_UNSUPPORTED;
#define B200_NORM_BWD(T, WT)                                                                                      \
  rc = mv <= 1   ? launch_norm_bwd<T, WT, 1>(layer_norm, dy, h, w, stats, dres_in, dx, dwp, dbp, rows, cols, grid, st) \
       : mv <= 2 ? launch_norm_bwd<T, WT, 2>(layer_norm, dy, h, w, stats, dres_in, dx, dwp, dbp, rows, cols, grid, st) \
                 : launch_norm_bwd<T, WT, 4>(layer_norm, dy, h, w, stats, dres_in, dx, dwp, dbp, rows, cols, grid, st)
  if (dtype == B200_DT_BF16 && wdtype == B200_DT_BF16) { B200_NORM_BWD(__nv_bfloat16, __nv_bfloat16); }
  else if (dtype == B200_DT_BF16 && wdtype == B200_DT_FP32) { B200_NORM_BWD(__nv_bfloat16, float); }
  else if (dtype == B200_DT_FP32 && wdtype == B200_DT_FP32) { B200_NORM_BWD(float, float); }
  else if (dtype == B200_DT_FP16 && wdtype == B200_DT_FP16) { B200_NORM_BWD(__half, __half); }
#undef B200_NORM_BWD
  if (rc) return rc;
  const int tb = 256, gb = ceil_div(cols, tb);
  if (dw) {
    if (wdtype == B200_DT_FP32) reduce_partials_kernel<float><<<gb, tb, 0, st>>>(dwp, (float*)dw, grid, cols, accumulate);
    else if (wdtype == B200_DT_BF16) reduce_partials_kernel<__nv_bfloat16><<<gb, tb, 0, st>>>(dwp, (__nv_bfloat16*)dw, grid, cols, accumulate);
    else reduce_partials_kernel<__half><<<gb, tb, 0, st>>>(dwp, (__half*)dw, grid, cols, accumulate);
  }
  if (db) {
    if (wdtype == B200_DT_FP32) reduce_partials_kernel<float><<<gb, tb, 0, st>>>(dbp, (float*)db, grid, cols, accumulate);
    else if (wdtype == B200_DT_BF16) reduce_partials_kernel<__nv_bfloat16><<<gb, tb, 0, st>>>(dbp, (__nv_bfloat16*)db, grid, cols, accumulate);
    else reduce_partials_kernel<__half><<<gb, tb, 0, st>>>(dbp, (__half*)db, grid, cols, accumulate);
  }
  B200_LAUNCH_CHECK();
  return 0;
}

// =================================================================================================
// b200_norm_bwd_noalloc — the same backward, for callers that must not allocate.
//
// Who that is: anything that reaches this library through the C ABI without an allocator it is
// allowed to use at call time — an inference/serving process that handed every free byte of HBM to
// its KV-cache pool at start-up, a plugin host or real-time loop that bans cudaMalloc after
// initialisation because it serialises the whole device, or a small C/C++ harness that simply has
// no caching allocator behind it (the Python side of this repository borrows torch's). The regular
// entry point asks such callers for a `scratch` buffer they have no good way to produce.
//
// This variant keeps the per-CTA dw/db partial rows in a fixed array that lives in the library
// image itself: kNoAllocScratchFloats floats = 8 MiB, present on every GPU that loads
// libb200ops.so from load until the process exits. To stay inside it the kernel runs with at most
// kNoAllocParts CTAs, and `cols` may not exceed kNoAllocMaxCols; anything larger is refused with
// B200_ERR_TOO_LARGE and a message on stderr — nothing is launched and nothing is allocated.
//
// Host code cannot hand the array's name to a kernel (on the host it is only a stand-in symbol),
// so the device address is looked up with cudaGetSymbolAddress, once per device, with that device
// current, the first time the entry point is called there; the result is cached. That first call
// therefore does a little extra driver work: make it before starting any stream capture.
//
// The array is shared by every call and keeps whatever the last call left in it. Nothing has to
// be cleared: each call rewrites every partial row its own reduction reads before reading it.
// The flip side is that two calls whose kernels may overlap on the GPU (different streams, or
// different host threads on the same device) race on the array — serialise them.
//
// No cudaMalloc / cudaFree / allocating library routine is called here, on any path.
// =================================================================================================
#include <mutex>

namespace b200 {
constexpr int kNoAllocMaxCols = 8192;
constexpr int kNoAllocParts = 128;
constexpr long long kNoAllocScratchFloats = 2ll * kNoAllocParts * kNoAllocMaxCols;  // dw rows, then db rows
static __device__ __align__(256) float g_norm_bwd_scratch[kNoAllocScratchFloats];

constexpr int kNoAllocMaxDevices = 64;
static float* g_norm_bwd_scratch_addr[kNoAllocMaxDevices] = {nullptr};
static std::mutex g_norm_bwd_scratch_mu;

// device address of the scratch array on the current device (looked up once per device)
static int norm_bwd_noalloc_scratch(float** out) {
  int dev = -1;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return (int)e;
  if (dev < 0 || dev >= kNoAllocMaxDevices) return B200_ERR_UNSUPPORTED;
  std::lock_guard<std::mutex> lock(g_norm_bwd_scratch_mu);
  if (g_norm_bwd_scratch_addr[dev] == nullptr) {
    float* p = nullptr;
    e = cudaGetSymbolAddress((void**)&p, g_norm_bwd_scratch);
    if (e != cudaSuccess) return (int)e;
    if (p == nullptr) return B200_ERR_UNSUPPORTED;
    g_norm_bwd_scratch_addr[dev] = p;
  }
  *out = g_norm_bwd_scratch_addr[dev];
  return 0;
}
}  // namespace b200

B200_API int b200_norm_bwd_noalloc_max_cols(void) { return b200::kNoAllocMaxCols; }

B200_API int b200_norm_bwd_noalloc(int layer_norm, const void* dy, const void* h, const void* w, const float* stats,
                                   const void* dres_in, void* dx, void* dw, void* db, int accumulate, int rows,
                                   int cols, int dtype, int wdtype, void* stream) {
  cudaStream_t st = (cudaStream_t)stream;
  const int V = dtype == B200_DT_FP32 ? 4 : 8;
  if (rows <= 0 || cols <= 0 || cols % V) return B200_ERR_BAD_SHAPE;
  if (cols > kNoAllocMaxCols) {
    fprintf(stderr,
            "b200_norm_bwd_noalloc: cols = %d exceeds the built-in scratch (max %d columns, %lld bytes); "
            "use b200_norm_bwd with caller-provided scratch instead\n",
            cols, kNoAllocMaxCols, kNoAllocScratchFloats * 4);
    return B200_ERR_TOO_LARGE;
  }
  const int nvec = cols / V;
  const int mv = ceil_div(nvec, kNormThreads);
  if (mv > 4) {
    // fp32 activations: a thread holds 4 columns per vector instead of 8, so the row limit of the kernel is half
    fprintf(stderr,
            "b200_norm_bwd_noalloc: cols = %d exceeds the limit for this activation type (%d columns for fp32, %d for "
            "bf16 / fp16); use b200_norm_bwd with caller-provided scratch instead\n",
            cols, kNoAllocMaxCols / 2, kNoAllocMaxCols);
    return B200_ERR_TOO_LARGE;
  }
  float* scratch = nullptr;
  int rc = norm_bwd_noalloc_scratch(&scratch);
  if (rc) return rc;
  const int grid = rows < kNoAllocParts ? rows : kNoAllocParts;
  float* dwp = dw ? scratch : nullptr;
  float* dbp = db ? scratch + (long long)kNoAllocParts * kNoAllocMaxCols : nullptr;
  rc = B200_ERR_UNSUPPORTED;
#define B200_NORM_BWD_NA(T, WT)                                                                                      \
  rc = mv <= 1   ? launch_norm_bwd<T, WT, 1>(layer_norm, dy, h, w, stats, dres_in, dx, dwp, dbp, rows, cols, grid, st) \
       : mv <= 2 ? launch_norm_bwd<T, WT, 2>(layer_norm, dy, h, w, stats, dres_in, dx, dwp, dbp, rows, cols, grid, st) \
                 : launch_norm_bwd<T, WT, 4>(layer_norm, dy, h, w, stats, dres_in, dx, dwp, dbp, rows, cols, grid, st)
  if (dtype == B200_DT_BF16 && wdtype == B200_DT_BF16) { B200_NORM_BWD_NA(__nv_bfloat16, __nv_bfloat16); }
  else if (dtype == B200_DT_BF16 && wdtype == B200_DT_FP32) { B200_NORM_BWD_NA(__nv_bfloat16, float); }
  else if (dtype == B200_DT_FP32 && wdtype == B200_DT_FP32) { B200_NORM_BWD_NA(float, float); }
  else if (dtype == B200_DT_FP16 && wdtype == B200_DT_FP16) { B200_NORM_BWD_NA(__half, __half); }
#undef B200_NORM_BWD_NA
  if (rc) return rc;
  const int tb = 256, gb = ceil_div(cols, tb);
  if (dw) {
    if (wdtype == B200_DT_FP32) reduce_partials_kernel<float><<<gb, tb, 0, st>>>(dwp, (float*)dw, grid, cols, accumulate);
    else if (wdtype == B200_DT_BF16) reduce_partials_kernel<__nv_bfloat16><<<gb, tb, 0, st>>>(dwp, (__nv_bfloat16*)dw, grid, cols, accumulate);
    else reduce_partials_kernel<__half><<<gb, tb, 0, st>>>(dwp, (__half*)dw, grid, cols, accumulate);
  }
  if (db) {
    if (wdtype == B200_DT_FP32) reduce_partials_kernel<float><<<gb, tb, 0, st>>>(dbp, (float*)db, grid, cols, accumulate);
    else if (wdtype == B200_DT_BF16) reduce_partials_kernel<__nv_bfloat16><<<gb, tb, 0, st>>>(dbp, (__nv_bfloat16*)db, grid, cols, accumulate);
    else reduce_partials_kernel<__half><<<gb, tb, 0, st>>>(dbp, (__half*)db, grid, cols, accumulate);
  }
  B200_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------------------------
// Sandwich norms around a 32-bit residual stream (pre- and post-sublayer RMSNorm, gain stored as an offset from `off`):
//     x   = res + rms(y) * (off + w_post)        (w_post == nullptr: x = res + y;  res_in == nullptr: res = 0)
//     h   = rms(x) * (off + w_next)              (w_next == nullptr: h is not written)
// x is written to the fp32 stream `res_out`; y and h have their own types (fp32 or 16-bit). One CTA per row, the row is
// kept in shared memory between the passes, all statistics and the stream itself are fp32.
// ---------------------------------------------------------------------------------------------
namespace b200 {
// `center` 1: both norms take the row's mean off first and divide by the root of the variance (a layer norm with a weight and
// no bias); the statistics are two passes over the row in shared memory (mean, then squared deviations). `y2`: a second branch
// with a weight of its own, normed by itself and added to the first.
template <typename TY, typename TH, typename WT>
__global__ void __launch_bounds__(kNormThreads)
sandwich_norm_kernel(const TY* __restrict__ y, const WT* __restrict__ w_post, const TY* __restrict__ y2,
                     const WT* __restrict__ w_post2, const float* __restrict__ res_in, float* __restrict__ res_out, const WT* __restrict__ w_next, TH* __restrict__ h,
                     int cols, float eps, float off, float mult, int center) {
  extern __shared__ float rowbuf[];
  __shared__ float red[32];
  const long long row = blockIdx.x;
  float ss = 0.f, s1 = 0.f;
  if (y) {
    const TY* yr = y + row * cols;
    for (int i = threadIdx.x; i < cols; i += blockDim.x) {
      const float v = to_f32<TY>(yr[i]);
      rowbuf[i] = v;
      ss += v * v;
      s1 += v;
    }
  } else {
    for (int i = threadIdx.x; i < cols; i += blockDim.x) rowbuf[i] = 0.f;
  }
  float r1 = 1.f, m1 = 0.f;
  if (w_post) {
    if (center) {
      m1 = block_sum(s1, red) / (float)cols;
      ss = 0.f;
      for (int i = threadIdx.x; i < cols; i += blockDim.x) { const float d = rowbuf[i] - m1; ss += d * d; }
    }
    ss = block_sum(ss, red);
    r1 = 1.f / sqrtf(ss / (float)cols + eps);
  }
  float* rowbuf2 = rowbuf + cols;                       // y2 only
  float r3 = 1.f;
  if (y2) {
    float s3 = 0.f;
    for (int i = threadIdx.x; i < cols; i += blockDim.x) {
      const float v = to_f32<TY>(y2[row * cols + i]);
      rowbuf2[i] = v;
      s3 += v * v;
    }
    s3 = block_sum(s3, red);
    r3 = 1.f / sqrtf(s3 / (float)cols + eps);
  }
  __syncthreads();
  float s2 = 0.f, t1 = 0.f;
  for (int i = threadIdx.x; i < cols; i += blockDim.x) {
    float v = rowbuf[i];
    if (w_post) v = (v - m1) * r1 * (off + to_f32<WT>(w_post[i]));
    if (y2) v = fmaf(rowbuf2[i] * r3, off + to_f32<WT>(w_post2[i]), v);
    v *= mult;
    if (res_in) v += res_in[row * cols + i];
    rowbuf[i] = v;
    if (res_out) res_out[row * cols + i] = v;
    s2 += v * v;
    t1 += v;
  }
  if (!w_next) {                                        // no norm follows: h, if asked for, is the stream in the next GEMM's dtype
    if (h)
      for (int i = threadIdx.x; i < cols; i += blockDim.x) h[row * cols + i] = from_f32<TH>(rowbuf[i]);
    return;
  }
  float m2 = 0.f;
  if (center) {
    m2 = block_sum(t1, red) / (float)cols;
    s2 = 0.f;
    for (int i = threadIdx.x; i < cols; i += blockDim.x) { const float d = rowbuf[i] - m2; s2 += d * d; }
  }
  s2 = block_sum(s2, red);
  const float r2 = 1.f / sqrtf(s2 / (float)cols + eps);
  for (int i = threadIdx.x; i < cols; i += blockDim.x)
    h[row * cols + i] = from_f32<TH>((rowbuf[i] - m2) * r2 * (off + to_f32<WT>(w_next[i])));
}

// four neighbouring elements as fp32, and back
template <typename T> __device__ __forceinline__ float4 load4(const T* p) {
  if constexpr (sizeof(T) == 4) {
    return *reinterpret_cast<const float4*>(p);
  } else {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const T* e = reinterpret_cast<const T*>(&r);
    return make_float4(to_f32<T>(e[0]), to_f32<T>(e[1]), to_f32<T>(e[2]), to_f32<T>(e[3]));
  }
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float4 v) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = v;
  } else {
    uint2 r;
    T* e = reinterpret_cast<T*>(&r);
    e[0] = from_f32<T>(v.x); e[1] = from_f32<T>(v.y); e[2] = from_f32<T>(v.z); e[3] = from_f32<T>(v.w);
    *reinterpret_cast<uint2*>(p) = r;
  }
}
__device__ __forceinline__ float dot4(const float4 v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))); }

// The RMS case of the kernel above for rows of whole groups of four columns: a thread keeps its NV groups in registers from the
// first load to the last store, so nothing passes through shared memory but the sums.
template <typename TY, typename TH, typename WT, int NV, bool TWO>
__global__ void __launch_bounds__(kNormThreads)
sandwich_norm_vec_kernel(const TY* __restrict__ y, const WT* __restrict__ w_post, const TY* __restrict__ y2,
                         const WT* __restrict__ w_post2, const float* __restrict__ res_in, float* __restrict__ res_out,
                         const WT* __restrict__ w_next, TH* __restrict__ h, int cols, float eps, float off, float mult) {
  __shared__ float red[32];
  const long long base = (long long)blockIdx.x * cols;
  float4 v[NV], v2[NV], x[NV];
  float ss = 0.f, s3 = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    v[j] = v2[j] = x[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= cols) continue;
    if (y) v[j] = load4<TY>(y + base + i);
    if (TWO) v2[j] = load4<TY>(y2 + base + i);
    if (res_in) x[j] = *reinterpret_cast<const float4*>(res_in + base + i);
  }
  float r1 = 1.f, r3 = 1.f;
  if (w_post) {
#pragma unroll
    for (int j = 0; j < NV; ++j) { ss += dot4(v[j]); if (TWO) s3 += dot4(v2[j]); }
    r1 = 1.f / sqrtf(block_sum(ss, red) / (float)cols + eps);
    if (TWO) r3 = 1.f / sqrtf(block_sum(s3, red) / (float)cols + eps);
  }
  float s2 = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i >= cols) continue;
    if (w_post) {
      const float4 w = load4<WT>(w_post + i);
      v[j] = make_float4(v[j].x * r1 * (off + w.x), v[j].y * r1 * (off + w.y), v[j].z * r1 * (off + w.z), v[j].w * r1 * (off + w.w));
    }
    if (TWO) {
      const float4 w = load4<WT>(w_post2 + i);
      v[j] = make_float4(fmaf(v2[j].x * r3, off + w.x, v[j].x), fmaf(v2[j].y * r3, off + w.y, v[j].y), fmaf(v2[j].z * r3, off + w.z, v[j].z),
                         fmaf(v2[j].w * r3, off + w.w, v[j].w));
    }
    x[j] = make_float4(fmaf(v[j].x, mult, x[j].x), fmaf(v[j].y, mult, x[j].y), fmaf(v[j].z, mult, x[j].z), fmaf(v[j].w, mult, x[j].w));
    if (res_out) *reinterpret_cast<float4*>(res_out + base + i) = x[j];
    s2 += dot4(x[j]);
  }
  float r2 = 1.f;
  if (w_next) r2 = 1.f / sqrtf(block_sum(s2, red) / (float)cols + eps);
  if (!h) return;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i >= cols) continue;
    if (w_next) {
      const float4 w = load4<WT>(w_next + i);
      x[j] = make_float4(x[j].x * r2 * (off + w.x), x[j].y * r2 * (off + w.y), x[j].z * r2 * (off + w.z), x[j].w * r2 * (off + w.w));
    }
    store4<TH>(h + base + i, x[j]);
  }
}

template <typename TY, typename TH, typename WT>
static int sandwich_launch(const void* y, const void* w_post, const void* y2, const void* w_post2, const float* res_in, float* res_out,
                           const void* w_next, void* h, long long rows, int cols, float eps, float off, float mult, int center, cudaStream_t st) {
  {
    auto al = [](const void* p_, size_t es) { return !(reinterpret_cast<uintptr_t>(p_) & (4 * es - 1)); };
    if (!center && cols % 4 == 0 && cols <= 16 * kNormThreads * 2 && al(y, sizeof(TY)) && al(y2, sizeof(TY)) && al(w_post, sizeof(WT)) &&
        al(w_post2, sizeof(WT)) && al(w_next, sizeof(WT)) && al(res_in, 4) && al(res_out, 4) && al(h, sizeof(TH))) {
      const int groups = (cols / 4 + kNormThreads - 1) / kNormThreads;
      int nt = (cols / 4 + groups - 1) / groups;          // no more threads than groups of columns
      nt = nt > kNormThreads ? kNormThreads : (nt + 31) / 32 * 32;
#define SWV(NV, TWO)                                                                                                          \
  sandwich_norm_vec_kernel<TY, TH, WT, NV, TWO><<<(unsigned)rows, nt, 0, st>>>((const TY*)y, (const WT*)w_post, (const TY*)y2,  \
      (const WT*)w_post2, res_in, res_out, (const WT*)w_next, (TH*)h, cols, eps, off, mult)
#define SWV_N(NV) do { if (y2) SWV(NV, true); else SWV(NV, false); } while (0)
      if (groups <= 1) SWV_N(1); else if (groups <= 2) SWV_N(2); else if (groups <= 4) SWV_N(4); else SWV_N(8);
#undef SWV_N
#undef SWV
      B200_LAUNCH_CHECK();
      return 0;
    }
  }
  const size_t smem = (size_t)cols * (y2 ? 2 : 1) * sizeof(float);
  auto kern = sandwich_norm_kernel<TY, TH, WT>;
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return B200_ERR_TOO_LARGE;
    B200_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  }
  kern<<<(unsigned)rows, kNormThreads, smem, st>>>((const TY*)y, (const WT*)w_post, (const TY*)y2, (const WT*)w_post2, res_in, res_out, (const WT*)w_next, (TH*)h,
                                                   cols, eps, off, mult, center);
  B200_LAUNCH_CHECK();
  return 0;
}
// y = a N(z) + b N(z^2) + c N(z^3) + e per row, N(v) = v / sqrt(mean(v^2) + eps): three power sums in one pass over the row,
// then a cubic in z per element. One CTA per row; V elements per load.
template <typename T, int V>
__global__ void __launch_bounds__(256)
poly_norm_kernel(const T* __restrict__ z, const float* __restrict__ act, T* __restrict__ y, int cols, float eps) {
  __shared__ float red[32];
  const T* zr = z + (long long)blockIdx.x * cols;
  T* yr = y + (long long)blockIdx.x * cols;
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  for (int i = threadIdx.x * V; i < cols; i += blockDim.x * V) {
    T raw[V];
    if (V > 1) *reinterpret_cast<uint4*>(raw) = *reinterpret_cast<const uint4*>(zr + i);
    else raw[0] = zr[i];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float v = to_f32<T>(raw[e]), v2 = v * v, v4 = v2 * v2;
      s1 += v2;
      s2 += v4;
      s3 = fmaf(v4, v2, s3);
    }
  }
  s1 = block_sum(s1, red);
  s2 = block_sum(s2, red);
  s3 = block_sum(s3, red);
  const float n = (float)cols;
  const float a = act[0] / sqrtf(s1 / n + eps), b = act[1] / sqrtf(s2 / n + eps), c = act[2] / sqrtf(s3 / n + eps), d = act[3];
  for (int i = threadIdx.x * V; i < cols; i += blockDim.x * V) {
    T raw[V];
    if (V > 1) *reinterpret_cast<uint4*>(raw) = *reinterpret_cast<const uint4*>(zr + i);
    else raw[0] = zr[i];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float v = to_f32<T>(raw[e]);
      raw[e] = from_f32<T>(fmaf(v, fmaf(v, fmaf(v, c, b), a), d));
    }
    if (V > 1) *reinterpret_cast<uint4*>(yr + i) = *reinterpret_cast<const uint4*>(raw);
    else yr[i] = raw[0];
  }
}
}  // namespace b200

B200_API int b200_sandwich_norm_2(const void* y, const void* w_post, const void* y2, const void* w_post2, const float* res_in,
                                  float* res_out, const void* w_next, void* h, long long rows, int cols, float eps, float off,
                                  float mult, int center, int y_dtype, int h_dtype, int w_dtype, void* stream) {
  using namespace b200;
  cudaStream_t st = (cudaStream_t)stream;
  if (rows <= 0) return 0;
  if (cols <= 0 || (y2 && (!y || !w_post || !w_post2 || center))) return B200_ERR_BAD_SHAPE;
  typedef __nv_bfloat16 bf;
#define SW(TY, TH, WT) return sandwich_launch<TY, TH, WT>(y, w_post, y2, w_post2, res_in, res_out, w_next, h, rows, cols, eps, off, mult, center, st)
  if (w_dtype == B200_DT_BF16) {
    if (y_dtype == B200_DT_FP32 && h_dtype == B200_DT_BF16) SW(float, bf, bf);
    if (y_dtype == B200_DT_BF16 && h_dtype == B200_DT_BF16) SW(bf, bf, bf);
    if (y_dtype == B200_DT_FP32 && h_dtype == B200_DT_FP32) SW(float, float, bf);
    if (y_dtype == B200_DT_BF16 && h_dtype == B200_DT_FP32) SW(bf, float, bf);
  } else if (w_dtype == B200_DT_FP32) {
    if (y_dtype == B200_DT_FP32 && h_dtype == B200_DT_FP32) SW(float, float, float);
    if (y_dtype == B200_DT_FP32 && h_dtype == B200_DT_BF16) SW(float, bf, float);
    if (y_dtype == B200_DT_BF16 && h_dtype == B200_DT_BF16) SW(bf, bf, float);
  }
#undef SW
  return B200_ERR_UNSUPPORTED;
}

B200_API int b200_sandwich_norm_c(const void* y, const void* w_post, const float* res_in, float* res_out, const void* w_next,
                                  void* h, long long rows, int cols, float eps, float off, float mult, int center, int y_dtype,
                                  int h_dtype, int w_dtype, void* stream) {
  return b200_sandwich_norm_2(y, w_post, nullptr, nullptr, res_in, res_out, w_next, h, rows, cols, eps, off, mult, center, y_dtype, h_dtype,
                              w_dtype, stream);
}

B200_API int b200_sandwich_norm(const void* y, const void* w_post, const float* res_in, float* res_out, const void* w_next,
                                void* h, long long rows, int cols, float eps, float off, float mult, int y_dtype, int h_dtype,
                                int w_dtype, void* stream) {
  return b200_sandwich_norm_c(y, w_post, res_in, res_out, w_next, h, rows, cols, eps, off, mult, 0, y_dtype, h_dtype, w_dtype,
                              stream);
}

B200_API int b200_poly_norm(const void* z, const float* act, void* y, long long rows, int cols, float eps, int dtype, void* stream) {
  using namespace b200;
  if (rows <= 0) return 0;
  if (cols <= 0) return B200_ERR_BAD_SHAPE;
  cudaStream_t st = (cudaStream_t)stream;
  const int V = dtype == B200_DT_FP32 ? 4 : 8;
  const bool vec = cols % V == 0 && !((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(y)) & 15);
#define PN(T, VV)                                                                                                            \
  do {                                                                                                                       \
    if (vec) poly_norm_kernel<T, VV><<<(unsigned)rows, 256, 0, st>>>((const T*)z, act, (T*)y, cols, eps);                     \
    else poly_norm_kernel<T, 1><<<(unsigned)rows, 256, 0, st>>>((const T*)z, act, (T*)y, cols, eps);                          \
  } while (0)
  if (dtype == B200_DT_BF16) PN(__nv_bfloat16, 8);
  else if (dtype == B200_DT_FP16) PN(__half, 8);
  else if (dtype == B200_DT_FP32) PN(float, 4);
  else return B200_ERR_UNSUPPORTED;
#undef PN
  B200_LAUNCH_CHECK();
  return 0;
}
