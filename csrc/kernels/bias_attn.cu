// Sliding-window attention whose scores carry a learned bias per distance and head and whose values are the keys
// (models/bias_attention.py).  Any sizes, bf16 or float32; scores, softmax and sums are float32.
//
//   bias_fwd_any_kernel      whole sequences: 16 queries per CTA, keys in tiles of 32 that serve both products
//   bias_decode_any_kernel   one query per row against a ring of cached keys; the token's own key comes from the projection
//                            and one head per key head stores it
//
// bias [heads, bias_ld] holds the bias of every distance inside the window.  flash_tc.cu and bias_decode_tc.cu hold the
// tensor-core forms.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <algorithm>

#include "../api.h"
#include "../common.cuh"

namespace ferrl {
namespace {

using bf16 = __nv_bfloat16;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kAnyQ = 16, kAnyK = 32;

template <typename T>
__global__ void __launch_bounds__(128) bias_fwd_any_kernel(BiasFwdArgs a) {
  extern __shared__ float sm[];
  const int D = a.D, KS = D + 1;
  float* sk = sm;                          // [kAnyK][D + 1]
  float* sq = sk + kAnyK * KS;             // [kAnyQ][D]
  float* so = sq + kAnyQ * D;              // [kAnyQ][D]
  float* sp = so + kAnyQ * D;              // [4 warps][kAnyK]
  const int h = blockIdx.y, b = blockIdx.z, q0 = blockIdx.x * kAnyQ;
  const int g = h / (a.Hq / a.Hkv);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* Q = static_cast<const T*>(a.q) + b * a.q_bs + static_cast<long long>(h) * D;
  const T* K = static_cast<const T*>(a.k) + b * a.k_bs + static_cast<long long>(g) * D;
  const float* bias = a.bias + static_cast<long long>(h) * a.bias_ld;
  for (int i = threadIdx.x; i < kAnyQ * D; i += 128) {
    const int r = i / D, c = i - r * D;
    sq[i] = q0 + r < a.S ? to_f(Q[(q0 + r) * a.q_ts + c]) : 0.f;
    so[i] = 0.f;
  }
  float m[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) { m[i] = -INFINITY; l[i] = 0.f; }
  const int last = min(q0 + kAnyQ, a.S) - 1;
  const int j_lo = max(0, q0 - a.window + 1) / kAnyK * kAnyK;
  for (int j0 = j_lo; j0 <= last; j0 += kAnyK) {
    __syncthreads();
    for (int i = threadIdx.x; i < kAnyK * D; i += 128) {
      const int r = i / D, c = i - r * D;
      sk[r * KS + c] = j0 + r < a.S ? to_f(K[(j0 + r) * a.k_ts + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int qi = 0; qi < 4; ++qi) {
      const int r = warp * 4 + qi, pos = q0 + r, key = j0 + lane;
      float s = -INFINITY;
      if (key <= pos && pos < a.S && pos - key < a.window) {
        s = 0.f;
        for (int c = 0; c < D; ++c) s += sq[r * D + c] * sk[lane * KS + c];
        s = s * a.scale + bias[pos - key];
      }
      const float mn = fmaxf(m[qi], warp_max(s));
      if (mn == -INFINITY) continue;       // warp-uniform: nothing visible yet
      const float p = s == -INFINITY ? 0.f : exp2f((s - mn) * kLog2e);
      const float corr = m[qi] == -INFINITY ? 0.f : exp2f((m[qi] - mn) * kLog2e);
      l[qi] = l[qi] * corr + warp_sum(p);
      m[qi] = mn;
      sp[warp * kAnyK + lane] = p;
      __syncwarp();
      for (int c = lane; c < D; c += 32) {
        float o = so[r * D + c] * corr;
        for (int k = 0; k < kAnyK; ++k) o += sp[warp * kAnyK + k] * sk[k * KS + c];
        so[r * D + c] = o;
      }
      __syncwarp();
    }
  }
#pragma unroll
  for (int qi = 0; qi < 4; ++qi) {
    const int r = warp * 4 + qi, pos = q0 + r;
    if (pos >= a.S) continue;
    const float inv = 1.f / l[qi];
    T* o = static_cast<T*>(a.out) + (static_cast<long long>(b) * a.S + pos) * a.Hq * D + static_cast<long long>(h) * D;
    for (int c = lane; c < D; c += 32) o[c] = from_f<T>(so[r * D + c] * inv);
  }
}

template <typename T>
__global__ void __launch_bounds__(128) bias_decode_any_kernel(BiasDecodeArgs a) {
  extern __shared__ float sm[];
  float* sq = sm;                       // [D]
  float* sn = sq + a.D;                 // [D] the token's own key
  float* so = sn + a.D;                 // [D]
  __shared__ float sp[128], red[32];
  pdl_trigger();
  const int h = blockIdx.x, b = blockIdx.y, D = a.D;
  const int rep = a.Hq / a.Hkv, g = h / rep;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  T* out = static_cast<T*>(a.out) + (static_cast<long long>(b) * a.Hq + h) * D;
  if (a.active && !a.active[b]) {       // a retired row attends to nothing and keeps its cache
    for (int i = threadIdx.x; i < D; i += 128) out[i] = from_f<T>(0.f);
    return;
  }
  const int pos = a.kv_len[b];
  const int n = min(pos + 1, a.slots), cur = pos % a.slots;
  const T* q = static_cast<const T*>(a.q) + b * a.ld_q + static_cast<long long>(h) * D;
  const T* kn = static_cast<const T*>(a.k) + b * a.ld_k + static_cast<long long>(g) * D;
  const long long row = static_cast<long long>(a.Hkv) * D;
  T* cache = static_cast<T*>(a.cache) + b * a.slots * row + static_cast<long long>(g) * D;
  const float* bias = a.bias + static_cast<long long>(h) * a.bias_ld;
  for (int i = threadIdx.x; i < D; i += 128) {
    const T kv = kn[i];
    sq[i] = to_f(q[i]);
    sn[i] = to_f(kv);
    so[i] = 0.f;
    if (h == g * rep) cache[cur * row + i] = kv;
  }
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < n; k0 += 128) {
    const int nk = min(128, n - k0);
    __syncthreads();
    for (int k = warp; k < nk; k += 4) {
      const int slot = k0 + k;
      const T* kr = cache + slot * row;
      float s = 0.f;
      for (int c = lane; c < D; c += 32) s += sq[c] * (slot == cur ? sn[c] : to_f(kr[c]));
      s = warp_sum(s);
      if (lane == 0) sp[k] = s * a.scale + bias[cur >= slot ? cur - slot : cur - slot + a.slots];
    }
    __syncthreads();
    const float s = static_cast<int>(threadIdx.x) < nk ? sp[threadIdx.x] : -INFINITY;
    const float mn = fmaxf(m, block_max(s, red));
    const float p = s == -INFINITY ? 0.f : exp2f((s - mn) * kLog2e);
    const float corr = m == -INFINITY ? 0.f : exp2f((m - mn) * kLog2e);
    l = l * corr + block_sum(p, red);
    m = mn;
    sp[threadIdx.x] = p;
    __syncthreads();
    for (int c = threadIdx.x; c < D; c += 128) {
      float o = so[c] * corr;
      for (int k = 0; k < nk; ++k) o += sp[k] * (k0 + k == cur ? sn[c] : to_f(cache[(k0 + k) * row + c]));
      so[c] = o;
    }
  }
  __syncthreads();
  const float inv = 1.f / l;
  for (int c = threadIdx.x; c < D; c += 128) out[c] = from_f<T>(so[c] * inv);
}

}  // namespace

const char* bias_fwd_any(const BiasFwdArgs& a, cudaStream_t s) {
  if (a.B == 0 || a.S == 0) return nullptr;
  const size_t smem = (static_cast<size_t>(kAnyK) * (a.D + 1) + 2 * kAnyQ * a.D + 4 * kAnyK) * 4;
  if (smem > 227 * 1024) return "bias_fwd: head size too large";
  if (!FERRL_ONCE_PER_DEVICE(
          cudaFuncSetAttribute(bias_fwd_any_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) == cudaSuccess &&
          cudaFuncSetAttribute(bias_fwd_any_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) == cudaSuccess))
    return "bias_fwd: cannot reserve shared memory";
  const dim3 grid((a.S + kAnyQ - 1) / kAnyQ, a.Hq, a.B);
  if (a.dtype == kF32) bias_fwd_any_kernel<float><<<grid, 128, smem, s>>>(a);
  else bias_fwd_any_kernel<bf16><<<grid, 128, smem, s>>>(a);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "bias_fwd launch failed";
}

const char* bias_decode_any(const BiasDecodeArgs& a, cudaStream_t s) {
  if (a.B == 0) return nullptr;
  const size_t smem = static_cast<size_t>(3) * a.D * 4;
  if (smem > 40 * 1024) return "bias_decode: head size too large";
  const dim3 grid(a.Hq, a.B);
  if (a.dtype == kF32) launch_pdl(bias_decode_any_kernel<float>, grid, dim3(128), smem, s, a);
  else launch_pdl(bias_decode_any_kernel<bf16>, grid, dim3(128), smem, s, a);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "bias_decode launch failed";
}

}  // namespace ferrl
