// State-space duality layers (models/mamba2.py): causal convolution, selective scan, one-token step, gated group norm.
//
// A head's state S is N x P float32.  Per token, with step size dt = softplus(raw + bias) and the group's B and C:
//
//   S <- exp(-exp(A_log) dt) S + dt B x^T        y = S^T C + D x
//
//   ssm_conv_kernel         whole sequences: y = silu(bias + sum_j w[c, j] x[t - K + 1 + j, c]), [B, L, C] in place of layout
//   ssm_scan_kernel         whole sequences, any sizes, all in float32: a warp owns four columns of S, eight lanes share a
//                           column's N entries in registers, tokens stream through shared memory (ssm_scan_tc.cu holds the
//                           chunked tensor-core form)
//   ssm_step_kernel         one token per row: convolution, step size, state update and output of one head; the
//                           convolution's inputs live in a ring of K slots, of which a step writes one that no head reads
//   gated_group_norm_kernel y silu(z), divided by the root mean square of each of its equal parts, times a weight
//
// Tokens at or past a sequence's length leave its state untouched.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <algorithm>

#include "../api.h"
#include "../common.cuh"
#include "../gemm/tc_common.cuh"
#include "vec.cuh"

namespace ferrl {
namespace {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + __expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(__expf(x)); }

// ------------------------------------------------------------------------------------------------ convolution
// A thread owns V channels and kRun consecutive tokens: the window slides through registers.
constexpr int kRun = 16;
template <typename T, int V> struct ConvIo;
template <typename T> struct ConvIo<T, 1> {
  static __device__ __forceinline__ void ld(const T* p, float* v) { v[0] = to_f(*p); }
  static __device__ __forceinline__ void st(T* p, const float* v) { *p = from_f<T>(v[0]); }
};
template <> struct ConvIo<bf16, 8> {
  static __device__ __forceinline__ void ld(const bf16* p, float* v) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(h[e]);
      v[2 * e] = f.x;
      v[2 * e + 1] = f.y;
    }
  }
  static __device__ __forceinline__ void st(bf16* p, const float* v) {
    uint4 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
    *reinterpret_cast<uint4*>(p) = u;
  }
};

// KT taps at compile time, or any number at run time (KT = 0, re-reading the window)
template <typename T, int V, int KT>
__global__ void ssm_conv_kernel(const T* __restrict__ x, long long x_bs, long long x_ts, const float* __restrict__ w,
                                const float* __restrict__ bias, T* __restrict__ y, int B, int L, int C, int K) {
  const int taps = KT > 0 ? KT : K;
  const int groups = C / V, runs = (L + kRun - 1) / kRun;
  const long long n = static_cast<long long>(B) * runs * groups;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int c = static_cast<int>(i % groups) * V;
    const long long br = i / groups;
    const int t0 = static_cast<int>(br % runs) * kRun, b = static_cast<int>(br / runs);
    const T* xp = x + b * x_bs + c;
    T* yp = y + (static_cast<long long>(b) * L + t0) * C + c;
    float bs[V];
#pragma unroll
    for (int e = 0; e < V; ++e) bs[e] = bias ? bias[c + e] : 0.f;
    if constexpr (KT > 0) {
      float wv[KT][V], win[KT][V];
      if constexpr (KT == 4) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const float4 f = *reinterpret_cast<const float4*>(w + static_cast<long long>(c + e) * 4);
          wv[0][e] = f.x; wv[1][e] = f.y; wv[2][e] = f.z; wv[3][e] = f.w;
        }
      } else {
#pragma unroll
        for (int j = 0; j < KT; ++j)
#pragma unroll
          for (int e = 0; e < V; ++e) wv[j][e] = w[static_cast<long long>(c + e) * KT + j];
      }
#pragma unroll
      for (int j = 1; j < KT; ++j) {          // win[j] holds token t0 - KT + j
        const int t = t0 - KT + j;
        if (t >= 0) {
          ConvIo<T, V>::ld(xp + t * x_ts, win[j]);
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) win[j][e] = 0.f;
        }
      }
      for (int r = 0; r < kRun && t0 + r < L; ++r) {
#pragma unroll
        for (int j = 0; j + 1 < KT; ++j)
#pragma unroll
          for (int e = 0; e < V; ++e) win[j][e] = win[j + 1][e];
        ConvIo<T, V>::ld(xp + (t0 + r) * x_ts, win[KT - 1]);
        float o[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          float acc = bs[e];
#pragma unroll
          for (int j = 0; j < KT; ++j) acc += wv[j][e] * win[j][e];
          o[e] = silu_f(acc);
        }
        ConvIo<T, V>::st(yp + static_cast<long long>(r) * C, o);
      }
    } else {
      for (int r = 0; r < kRun && t0 + r < L; ++r) {
        float o[V];
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = bs[e];
        for (int j = 0; j < taps; ++j) {
          const int t = t0 + r - (taps - 1) + j;
          if (t < 0) continue;
          float v[V];
          ConvIo<T, V>::ld(xp + t * x_ts, v);
#pragma unroll
          for (int e = 0; e < V; ++e) o[e] += w[static_cast<long long>(c + e) * taps + j] * v[e];
        }
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = silu_f(o[e]);
        ConvIo<T, V>::st(yp + static_cast<long long>(r) * C, o);
      }
    }
  }
}

template <typename T, int V>
void launch_conv(const void* x, long long x_bs, long long x_ts, const float* w, const float* bias, void* y, int B, int L, int C, int K,
                 cudaStream_t s) {
  const long long n = static_cast<long long>(B) * ((L + kRun - 1) / kRun) * (C / V);
  const unsigned grid = static_cast<unsigned>(std::min<long long>((n + 127) / 128, 1 << 20));
  const T* xp = static_cast<const T*>(x);
  T* yp = static_cast<T*>(y);
  switch (K) {
    case 2: ssm_conv_kernel<T, V, 2><<<grid, 128, 0, s>>>(xp, x_bs, x_ts, w, bias, yp, B, L, C, K); break;
    case 3: ssm_conv_kernel<T, V, 3><<<grid, 128, 0, s>>>(xp, x_bs, x_ts, w, bias, yp, B, L, C, K); break;
    case 4:
      if ((reinterpret_cast<uintptr_t>(w) & 15) == 0) {
        ssm_conv_kernel<T, V, 4><<<grid, 128, 0, s>>>(xp, x_bs, x_ts, w, bias, yp, B, L, C, K);
        break;
      }
      [[fallthrough]];
    default: ssm_conv_kernel<T, V, 0><<<grid, 128, 0, s>>>(xp, x_bs, x_ts, w, bias, yp, B, L, C, K); break;
  }
}

// ------------------------------------------------------------------------------------------------ scan, any sizes
constexpr int kTile = 16, kCols = 32;      // tokens staged together, columns of S per CTA
template <typename T, int Q>               // Q: float4 groups of S entries per lane; N <= 32 Q
__global__ void __launch_bounds__(256) ssm_scan_kernel(SsmScanArgs a) {
  constexpr int NP = 32 * Q;
  extern __shared__ __align__(16) float sm[];
  float* sB = sm;                          // [kTile][NP]
  float* sC = sB + kTile * NP;             // [kTile][NP]
  float* sx = sC + kTile * NP;             // [kTile][kCols]
  float* sy = sx + kTile * kCols;          // [kTile][kCols]
  float* sdt = sy + kTile * kCols;         // [kTile]
  float* sda = sdt + kTile;                // [kTile]
  const int p0 = blockIdx.x * kCols, h = blockIdx.y, b = blockIdx.z;
  const int g = h / (a.H / a.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ng = lane & 7, col = warp * 4 + (lane >> 3);
  const int len = a.lens ? static_cast<int>(min(max(a.lens[b], 0ll), static_cast<long long>(a.T))) : a.T;
  const T* X = static_cast<const T*>(a.x) + b * a.bs + static_cast<long long>(h) * a.P + p0;
  const T* Bp = static_cast<const T*>(a.Bm) + b * a.bs + static_cast<long long>(g) * a.N;
  const T* Cp = static_cast<const T*>(a.Cm) + b * a.bs + static_cast<long long>(g) * a.N;
  const T* DT = static_cast<const T*>(a.dt) + b * a.dt_bs + h;
  T* Y = static_cast<T*>(a.y) + b * static_cast<long long>(a.T) * a.H * a.P + static_cast<long long>(h) * a.P + p0;
  const float A = -__expf(a.A_log[h]), D = a.D[h], dtb = a.dt_bias[h];
  const int cols = min(kCols, a.P - p0);
  float S[Q][4];
#pragma unroll
  for (int q = 0; q < Q; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) S[q][e] = 0.f;
  for (int t0 = 0; t0 < a.T; t0 += kTile) {
    const int nt = min(kTile, a.T - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < kTile * NP; i += 256) {
      const int t = i / NP, n = i - t * NP;
      const bool ok = t < nt && n < a.N;
      sB[i] = ok ? to_f(Bp[(t0 + t) * a.ts + n]) : 0.f;
      sC[i] = ok ? to_f(Cp[(t0 + t) * a.ts + n]) : 0.f;
    }
    for (int i = threadIdx.x; i < kTile * kCols; i += 256) {
      const int t = i / kCols, c = i - t * kCols;
      sx[i] = t < nt && c < cols ? to_f(X[(t0 + t) * a.ts + c]) : 0.f;
    }
    if (threadIdx.x < kTile) {
      float d = 0.f;
      if (static_cast<int>(threadIdx.x) < nt && t0 + static_cast<int>(threadIdx.x) < len)
        d = softplus_f(to_f(DT[(t0 + threadIdx.x) * a.dt_ts]) + dtb);
      sdt[threadIdx.x] = d;
      sda[threadIdx.x] = __expf(A * d);
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float da = sda[t], xv = sx[t * kCols + col], dx = sdt[t] * xv;
      float acc = 0.f;
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const float4 bv = *reinterpret_cast<const float4*>(sB + t * NP + q * 32 + ng * 4);
        const float4 cv = *reinterpret_cast<const float4*>(sC + t * NP + q * 32 + ng * 4);
        S[q][0] = S[q][0] * da + bv.x * dx;
        S[q][1] = S[q][1] * da + bv.y * dx;
        S[q][2] = S[q][2] * da + bv.z * dx;
        S[q][3] = S[q][3] * da + bv.w * dx;
        acc += S[q][0] * cv.x + S[q][1] * cv.y + S[q][2] * cv.z + S[q][3] * cv.w;
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      acc += __shfl_xor_sync(0xffffffffu, acc, 4);
      if (ng == 0) sy[t * kCols + col] = acc + D * xv;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * kCols; i += 256) {
      const int t = i / kCols, c = i - t * kCols;
      if (c < cols) Y[static_cast<long long>(t0 + t) * a.H * a.P + c] = from_f<T>(sy[i]);
    }
  }
  if (a.state && col < cols) {
    float* So = a.state + (static_cast<long long>(b) * a.H + h) * a.N * a.P + p0 + col;
#pragma unroll
    for (int q = 0; q < Q; ++q)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = q * 32 + ng * 4 + e;
        if (n < a.N) So[static_cast<long long>(n) * a.P] = S[q][e];
      }
  }
}

template <typename T, int Q>
const char* launch_scan(const SsmScanArgs& a, cudaStream_t s) {
  const size_t smem = (static_cast<size_t>(2) * kTile * 32 * Q + 2 * kTile * kCols + 2 * kTile) * 4;
  auto k = ssm_scan_kernel<T, Q>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024) == cudaSuccess))
    return "ssm_scan: cannot reserve shared memory";
  k<<<dim3((a.P + kCols - 1) / kCols, a.H, a.B), 256, smem, s>>>(a);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "ssm_scan launch failed";
}
template <typename T>
const char* launch_scan_n(const SsmScanArgs& a, cudaStream_t s) {
  if (a.N <= 32) return launch_scan<T, 1>(a, s);
  if (a.N <= 64) return launch_scan<T, 2>(a, s);
  if (a.N <= 128) return launch_scan<T, 4>(a, s);
  if (a.N <= 256) return launch_scan<T, 8>(a, s);
  if (a.N <= 512) return launch_scan<T, 16>(a, s);
  return "ssm_scan: state of more than 512 entries per column";
}

// ------------------------------------------------------------------------------------------------ one token
// One CTA per (head, row).  BULK: the head's matrix is fetched with one bulk copy while the convolution runs, updated in
// shared memory and written back with another, so that several CTAs keep a streaming multiprocessor's memory requests in
// flight without holding them in registers; otherwise it is updated in place in global memory.
constexpr int kStepThreads = 128;
struct StepSmem { int x, B, C, part, bar, bytes, RG; };      // offsets in floats behind the matrix, total bytes
__host__ __device__ inline StepSmem step_smem(int P, int N, int V, bool bulk) {
  StepSmem m;
  m.RG = kStepThreads / (P / V) > 1 ? kStepThreads / (P / V) : 1;
  m.x = bulk ? N * P : 0;
  m.B = m.x + (P + 3) / 4 * 4;
  m.C = m.B + N;
  m.part = m.B + (2 * N + 3) / 4 * 4;
  m.bar = m.part + (m.RG * P + 3) / 4 * 4;
  m.bytes = m.bar * 4 + 16;
  return m;
}

// KT taps at compile time (the inputs of several channels are then requested together), or any number (KT = 0)
template <typename T, int V, bool BULK, int KT>
__global__ void __launch_bounds__(kStepThreads) ssm_step_kernel(SsmStepArgs a) {
  extern __shared__ __align__(128) float sm[];
  __shared__ float s_dt;
  pdl_trigger();
  const StepSmem lay = step_smem(a.P, a.N, V, BULK);
  const int h = blockIdx.x, b = blockIdx.y;
  const int rep = a.H / a.G, g = h / rep, inner = a.H * a.P, cgn = a.P / V;
  float *sx = sm + lay.x, *sB = sm + lay.B, *sC = sm + lay.C, *part = sm + lay.part;
  uint64_t* bar = reinterpret_cast<uint64_t*>(sm + lay.bar);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bar + 1);
  float* Sg = a.state + (static_cast<long long>(b) * a.H + h) * a.N * a.P;
  pdl_wait();
  T* y = static_cast<T*>(a.y) + static_cast<long long>(b) * inner + static_cast<long long>(h) * a.P;
  if (a.active && !a.active[b]) {                   // a retired row: nothing of its state moves
    for (int i = threadIdx.x; i < a.P; i += kStepThreads) y[i] = from_f<T>(0.f);
    return;
  }
  if constexpr (BULK) {
    if (threadIdx.x == 0) {
      tc::mbar_init(bar, 1);
      *abort_flag = 0;
      asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
      tc::mbar_expect_tx(bar, a.N * a.P * 4);
      tc::bulk_load(sm, Sg, a.N * a.P * 4, bar);
    }
  }
  const int pos = a.kv_len[b];
  const int cur = pos % a.K;
  const T* xr = static_cast<const T*>(a.x) + b * a.ld_x;            // this token's [x | B | C] channels
  T* ring = static_cast<T*>(a.ring) + static_cast<long long>(b) * a.K * a.C;
  const int n_ch = a.P + 2 * a.N;
  auto channel = [&](int i) {
    return i < a.P ? h * a.P + i : (i < a.P + a.N ? inner + g * a.N + (i - a.P) : inner + a.G * a.N + g * a.N + (i - a.P - a.N));
  };
  auto put = [&](int i, int c, T now, float acc) {
    if (i < a.P || h == g * rep) ring[static_cast<long long>(cur) * a.C + c] = now;
    sx[i < a.P ? i : i + lay.B - lay.x - a.P] = to_f(from_f<T>(silu_f(acc)));   // rounded as the convolution of whole sequences stores it
  };
  // token pos - j sits j slots behind the current one
  auto slot = [&](int j) { return static_cast<long long>(cur - j < 0 ? cur - j + a.K : cur - j) * a.C; };
  if constexpr (KT > 0) {
    constexpr int CH = 3;
    for (int i0 = threadIdx.x; i0 < n_ch; i0 += CH * kStepThreads) {
      T now[CH], past[CH][KT - 1];
      float w[CH][KT], acc[CH];
#pragma unroll
      for (int u = 0; u < CH; ++u) {
        const int i = i0 + u * kStepThreads, c = channel(i < n_ch ? i : i0);
        now[u] = xr[c];
        acc[u] = a.conv_b ? a.conv_b[c] : 0.f;
#pragma unroll
        for (int j = 0; j < KT; ++j) w[u][j] = a.conv_w[static_cast<long long>(c) * KT + j];
#pragma unroll
        for (int j = 1; j < KT; ++j) past[u][j - 1] = ring[slot(j) + c];
      }
#pragma unroll
      for (int u = 0; u < CH; ++u) {
        const int i = i0 + u * kStepThreads;
        if (i >= n_ch) break;
#pragma unroll
        for (int j = KT - 1; j >= 1; --j) acc[u] += w[u][KT - 1 - j] * (j <= pos ? to_f(past[u][j - 1]) : 0.f);
        acc[u] += w[u][KT - 1] * to_f(now[u]);
        put(i, channel(i), now[u], acc[u]);
      }
    }
  } else {
    for (int i = threadIdx.x; i < n_ch; i += kStepThreads) {
      const int c = channel(i);
      const T now = xr[c];
      float acc = a.conv_b ? a.conv_b[c] : 0.f;
      for (int j = 1; j < a.K; ++j) acc += a.conv_w[static_cast<long long>(c) * a.K + a.K - 1 - j] * (j <= pos ? to_f(ring[slot(j) + c]) : 0.f);
      acc += a.conv_w[static_cast<long long>(c) * a.K + a.K - 1] * to_f(now);
      put(i, c, now, acc);
    }
  }
  if (threadIdx.x == 0) s_dt = softplus_f(to_f(static_cast<const T*>(a.dt)[b * a.ld_dt + h]) + a.dt_bias[h]);
  __syncthreads();
  const float dt = s_dt, da = __expf(-__expf(a.A_log[h]) * dt);
  bool ok = true;
  if constexpr (BULK) ok = tc::mbar_wait(bar, 0, abort_flag, a.status, kStatusWaitTimeoutProducer);
  float* S = BULK ? sm : Sg;
  if (ok) {
    for (int item = threadIdx.x; item < lay.RG * cgn; item += kStepThreads) {
      const int rg = item / cgn, c = (item - rg * cgn) * V;
      Vec<V> acc, dx = ld<V>(sx + c);
#pragma unroll
      for (int e = 0; e < V; ++e) { acc.v[e] = 0.f; dx.v[e] *= dt; }
#pragma unroll 4
      for (int n = rg; n < a.N; n += lay.RG) {
        Vec<V> v = ld<V>(S + static_cast<long long>(n) * a.P + c);
        const float bn = sB[n], cn = sC[n];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          v.v[e] = v.v[e] * da + bn * dx.v[e];
          acc.v[e] += v.v[e] * cn;
        }
        st<V>(S + static_cast<long long>(n) * a.P + c, v);
      }
      st<V>(part + rg * a.P + c, acc);
    }
    if constexpr (BULK) tc::fence_async_smem();     // the bulk copy below reads what these threads wrote
  }
  if (__syncthreads_or(!ok)) {
    if constexpr (BULK) {
      for (int i = 0; i < 64; ++i) __nanosleep(10000);   // let the copy in flight land before shared memory goes away
    }
    return;
  }
  if constexpr (BULK) {
    if (threadIdx.x == 0) tc::bulk_store(Sg, sm, a.N * a.P * 4);
  }
  for (int i = threadIdx.x; i < a.P; i += kStepThreads) {
    float o = 0.f;
    for (int r = 0; r < lay.RG; ++r) o += part[r * a.P + i];
    y[i] = from_f<T>(o + a.D[h] * sx[i]);
  }
  if constexpr (BULK) {
    if (threadIdx.x == 0) tc::bulk_store_drain();
  }
}

template <typename T, int V, bool BULK, int KT>
const char* launch_step_taps(const SsmStepArgs& a, cudaStream_t s) {
  const int bytes = step_smem(a.P, a.N, V, BULK).bytes;
  if (bytes > 226 * 1024) return "ssm_step: head too large";
  auto k = ssm_step_kernel<T, V, BULK, KT>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024) == cudaSuccess))
    return "ssm_step: cannot reserve shared memory";
  launch_pdl(k, dim3(a.H, a.B), dim3(kStepThreads), bytes, s, a);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "ssm_step launch failed";
}
template <typename T, int V, bool BULK>
const char* launch_step(const SsmStepArgs& a, cudaStream_t s) {
  return a.K == 4 ? launch_step_taps<T, V, BULK, 4>(a, s) : launch_step_taps<T, V, BULK, 0>(a, s);
}
template <typename T>
const char* launch_step_any(const SsmStepArgs& a, cudaStream_t s) {
  if (a.P % 4 || (reinterpret_cast<uintptr_t>(a.state) & 15)) return launch_step<T, 1, false>(a, s);
  // a bulk-staged matrix should leave room for a few CTAs on an SM
  if (step_smem(a.P, a.N, 4, true).bytes <= 72 * 1024) return launch_step<T, 4, true>(a, s);
  return launch_step<T, 4, false>(a, s);
}

// ------------------------------------------------------------------------------------------------ gated norm
template <typename T, int V>
__global__ void gated_group_norm_kernel(const T* __restrict__ y, long long ld_y, const T* __restrict__ z, long long ld_z,
                                        const float* __restrict__ w, T* __restrict__ out, int W, int part, float eps) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const long long row = blockIdx.y;
  const int c0 = blockIdx.x * part;
  const T* yr = y + row * ld_y + c0;
  const T* zr = z + row * ld_z + c0;
  float sq = 0.f;
  for (int c = threadIdx.x * V; c < part; c += blockDim.x * V) {
    Vec<V> v = ld<V>(yr + c);
    const Vec<V> zv = ld<V>(zr + c);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      v.v[e] *= silu_f(zv.v[e]);
      sq += v.v[e] * v.v[e];
    }
    st<V>(sm + c, v);
  }
  const float r = 1.f / sqrtf(block_sum(sq, red) / static_cast<float>(part) + eps);
  for (int c = threadIdx.x * V; c < part; c += blockDim.x * V) {
    Vec<V> v = ld<V>(sm + c);
    const Vec<V> wv = ld<V>(w + c0 + c);
#pragma unroll
    for (int e = 0; e < V; ++e) v.v[e] *= r * wv.v[e];
    st<V>(out + row * W + c0 + c, v);
  }
}

template <typename T>
const char* launch_group_norm(const void* y, long long ld_y, const void* z, long long ld_z, const float* w, void* out, long long rows, int W,
                              int groups, float eps, cudaStream_t s) {
  const int part = W / groups;
  auto al = [](const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const bool vec = part % 4 == 0 && ld_y % 4 == 0 && ld_z % 4 == 0 && W % 4 == 0 && al(y, sizeof(T) * 4) && al(z, sizeof(T) * 4) && al(w, 16) &&
                   al(out, sizeof(T) * 4);
  const int threads = std::min(256, std::max(32, (part / (vec ? 4 : 1) + 31) / 32 * 32));
  auto k4 = gated_group_norm_kernel<T, 4>;
  auto k1 = gated_group_norm_kernel<T, 1>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(k4, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess &&
                             cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess))
    return "gated_group_norm: cannot reserve shared memory";
  for (long long r0 = 0; r0 < rows; r0 += 65535) {      // rows ride in the grid's y dimension
    const unsigned n = static_cast<unsigned>(std::min<long long>(65535, rows - r0));
    launch_pdl(vec ? k4 : k1, dim3(groups, n), dim3(threads), static_cast<size_t>(part) * 4, s, static_cast<const T*>(y) + r0 * ld_y, ld_y,
               static_cast<const T*>(z) + r0 * ld_z, ld_z, w, static_cast<T*>(out) + r0 * W, W, part, eps);
    count_launch();
  }
  return cudaGetLastError() == cudaSuccess ? nullptr : "gated_group_norm launch failed";
}

}  // namespace

const char* ssm_conv(int dtype, const void* x, long long x_bs, long long x_ts, const float* w, const float* bias, void* y, int B, int L, int C,
                     int K, cudaStream_t s) {
  if (B == 0 || L == 0 || C == 0) return nullptr;
  if (K < 1) return "ssm_conv: at least one tap";
  const bool vec = dtype == kBF16 && C % 8 == 0 && x_bs % 8 == 0 && x_ts % 8 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(y) & 15) == 0;
  if (dtype == kF32) launch_conv<float, 1>(x, x_bs, x_ts, w, bias, y, B, L, C, K, s);
  else if (vec) launch_conv<bf16, 8>(x, x_bs, x_ts, w, bias, y, B, L, C, K, s);
  else launch_conv<bf16, 1>(x, x_bs, x_ts, w, bias, y, B, L, C, K, s);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "ssm_conv launch failed";
}

const char* ssm_scan(const SsmScanArgs& a, cudaStream_t s) {
  if (a.B == 0) return nullptr;
  return a.dtype == kF32 ? launch_scan_n<float>(a, s) : launch_scan_n<bf16>(a, s);
}

const char* ssm_step(const SsmStepArgs& a, cudaStream_t s) {
  if (a.B == 0) return nullptr;
  return a.dtype == kF32 ? launch_step_any<float>(a, s) : launch_step_any<bf16>(a, s);
}

const char* gated_group_norm(int dtype, const void* y, long long ld_y, const void* z, long long ld_z, const float* w, void* out, long long rows,
                             int W, int groups, float eps, cudaStream_t s) {
  if (rows == 0) return nullptr;
  if (groups < 1 || W % groups) return "gated_group_norm: the parts must be equal";
  if (static_cast<long long>(W / groups) * 4 > 200 * 1024) return "gated_group_norm: part too wide";
  return dtype == kF32 ? launch_group_norm<float>(y, ld_y, z, ld_z, w, out, rows, W, groups, eps, s)
                       : launch_group_norm<bf16>(y, ld_y, z, ld_z, w, out, rows, W, groups, eps, s);
}

}  // namespace ferrl
