// Hyper-connections: `ns` residual streams per token, float32, of which every sublayer reads one mixture and to which it
// gives its output back through learned coefficients.  One kernel closes a sublayer and opens the next:
//
//   x_t <- sum_s mix[s, t] x_s + out[t] y          (y absent: the streams stay as they are)
//   u    = sum_s in[s] x_s                         (in absent: the plain sum)
//   h    = u / sqrt(mean(u^2) + eps) * (1 + w) * scale, in the compute dtype
//
// One CTA per token; the streams are read and written once, u stays in shared memory between the passes.
// embed_streams_kernel starts the streams: an embedding row plus a row of a position table, ns times.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <algorithm>

#include "../api.h"
#include "../common.cuh"
#include "vec.cuh"

namespace ferrl {
namespace {

using bf16 = __nv_bfloat16;
constexpr int kMaxStreams = 32;

// NS streams at compile time, or up to kMaxStreams of them at run time (NS = 0)
template <typename TY, typename TC, int NS, int V>
__global__ void __launch_bounds__(512) hyper_norm_kernel(HyperNormArgs a) {
  extern __shared__ __align__(16) float sm_u[];
  __shared__ float red[32];
  __shared__ float s_mix[kMaxStreams * kMaxStreams], s_out[kMaxStreams], s_in[kMaxStreams];
  constexpr int CAP = NS > 0 ? NS : kMaxStreams, UN = NS > 0 ? NS : 1;
  const int ns = NS > 0 ? NS : a.ns;
  pdl_trigger();
  // the coefficients are weights: no kernel of the step writes them
  for (int i = threadIdx.x; i < ns * ns; i += blockDim.x) s_mix[i] = a.y ? a.mix[i] : 0.f;
  for (int i = threadIdx.x; i < ns; i += blockDim.x) {
    s_out[i] = a.y ? a.out[i] : 0.f;
    s_in[i] = a.in ? a.in[i] : 1.f;
  }
  pdl_wait();
  __syncthreads();
  const long long row = blockIdx.x;
  float* x = a.x + row * ns * a.W;
  const TY* y = a.y ? static_cast<const TY*>(a.y) + row * a.ld_y : nullptr;
  float sq = 0.f;
  for (int c = threadIdx.x * V; c < a.W; c += blockDim.x * V) {
    Vec<V> xs[CAP];
#pragma unroll(UN)
    for (int s = 0; s < CAP; ++s)
      if (NS > 0 || s < ns) xs[s] = ld<V>(x + static_cast<long long>(s) * a.W + c);
    Vec<V> u;
#pragma unroll
    for (int e = 0; e < V; ++e) u.v[e] = 0.f;
    if (y) {
      const Vec<V> yv = ld<V>(y + c);
#pragma unroll(UN)
      for (int t = 0; t < CAP; ++t) {
        if (NS == 0 && t >= ns) break;
        Vec<V> n;
#pragma unroll
        for (int e = 0; e < V; ++e) n.v[e] = s_out[t] * yv.v[e];
#pragma unroll(UN)
        for (int s = 0; s < CAP; ++s)
          if (NS > 0 || s < ns) {
#pragma unroll
            for (int e = 0; e < V; ++e) n.v[e] += s_mix[s * ns + t] * xs[s].v[e];
          }
        if (a.store) st<V>(x + static_cast<long long>(t) * a.W + c, n);
#pragma unroll
        for (int e = 0; e < V; ++e) u.v[e] += s_in[t] * n.v[e];
      }
    } else {
#pragma unroll(UN)
      for (int s = 0; s < CAP; ++s)
        if (NS > 0 || s < ns) {
#pragma unroll
          for (int e = 0; e < V; ++e) u.v[e] += s_in[s] * xs[s].v[e];
        }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) sq += u.v[e] * u.v[e];
    st<V>(sm_u + c, u);
  }
  const float r = a.scale / sqrtf(block_sum(sq, red) / static_cast<float>(a.W) + a.eps);
  TC* h = static_cast<TC*>(a.h) + row * a.W;
  for (int c = threadIdx.x * V; c < a.W; c += blockDim.x * V) {
    Vec<V> u = ld<V>(sm_u + c);
    const Vec<V> w = ld<V>(a.w + c);
#pragma unroll
    for (int e = 0; e < V; ++e) u.v[e] = u.v[e] * r * (1.f + w.v[e]);
    st<V>(h + c, u);
  }
}

template <typename TY, typename TC, int NS>
const char* launch_ns(const HyperNormArgs& a, cudaStream_t s) {
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = NS > 0 && a.W % 4 == 0 && a.ld_y % 4 == 0 && al16(a.x) && (reinterpret_cast<uintptr_t>(a.y) & (sizeof(TY) * 4 - 1)) == 0 &&
                   al16(a.w) && al16(a.h);
  const int per = vec ? 4 : 1;
  const int cap = NS == 0 || a.rows >= 1024 ? 256 : 512;      // wide blocks for few rows, within the register file
  const int threads = std::min(cap, std::max(64, (a.W / per + 31) / 32 * 32));
  auto k4 = hyper_norm_kernel<TY, TC, NS, NS == 0 ? 1 : 4>;
  auto k1 = hyper_norm_kernel<TY, TC, NS, 1>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(k4, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess &&
                             cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess))
    return "hyper_norm: cannot reserve shared memory";
  launch_pdl(vec ? k4 : k1, dim3(static_cast<unsigned>(a.rows)), dim3(threads), static_cast<size_t>(a.W) * 4, s, a);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "hyper_norm launch failed";
}

template <typename TY, typename TC>
const char* launch_types(const HyperNormArgs& a, cudaStream_t s) {
  switch (a.ns) {
    case 1: return launch_ns<TY, TC, 1>(a, s);
    case 2: return launch_ns<TY, TC, 2>(a, s);
    case 3: return launch_ns<TY, TC, 3>(a, s);
    case 4: return launch_ns<TY, TC, 4>(a, s);
    default: return launch_ns<TY, TC, 0>(a, s);
  }
}

template <typename T, int V>
__global__ void embed_streams_kernel(const long long* __restrict__ ids, const T* __restrict__ table, const float* __restrict__ pe,
                                     const long long* __restrict__ pos, const int* __restrict__ kv_len, long long S,
                                     float* __restrict__ out, int W, int ns, long long vocab, long long max_pos) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  long long id = ids[t];
  if (id < 0 || id >= vocab) id = 0;   // never index out of the tables
  long long p = kv_len ? kv_len[t] : pos[t % S];
  p = min(max(p, 0ll), max_pos - 1);
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
    Vec<V> v = ld<V>(table + id * W + c);
    const Vec<V> e = ld<V>(pe + p * W + c);
#pragma unroll
    for (int i = 0; i < V; ++i) v.v[i] += e.v[i];
    for (int s = 0; s < ns; ++s) st<V>(out + (t * ns + s) * W + c, v);
  }
}

}  // namespace

const char* hyper_norm(const HyperNormArgs& a, cudaStream_t s) {
  if (a.rows == 0) return nullptr;
  if (a.ns < 1 || a.ns > kMaxStreams) return "hyper_norm: 1 to 32 streams";
  if (static_cast<long long>(a.W) * 4 > 200 * 1024) return "hyper_norm: row too wide";
  if (a.h_dtype == kF32 && a.y_dtype == kF32) return launch_types<float, float>(a, s);
  if (a.h_dtype == kBF16 && a.y_dtype == kBF16) return launch_types<bf16, bf16>(a, s);
  return "hyper_norm: unsupported dtype combination";
}

const char* embed_streams(int dtype, const long long* ids, const void* table, const float* pe, const long long* pos, const int* kv_len,
                          long long S, float* out, long long n_tok, int W, int ns, long long vocab, long long max_pos, cudaStream_t s) {
  if (n_tok == 0) return nullptr;
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = W % 4 == 0 && al16(table) && al16(pe) && al16(out);
  const dim3 grid(static_cast<unsigned>(n_tok)), block(std::min(256, std::max(32, (W / (vec ? 4 : 1) + 31) / 32 * 32)));
  if (dtype == kF32) {
    auto k = vec ? embed_streams_kernel<float, 4> : embed_streams_kernel<float, 1>;
    launch_pdl(k, grid, block, 0, s, ids, static_cast<const float*>(table), pe, pos, kv_len, S, out, W, ns, vocab, max_pos);
  } else {
    auto k = vec ? embed_streams_kernel<bf16, 4> : embed_streams_kernel<bf16, 1>;
    launch_pdl(k, grid, block, 0, s, ids, static_cast<const bf16*>(table), pe, pos, kv_len, S, out, W, ns, vocab, max_pos);
  }
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "embed_streams launch failed";
}

}  // namespace ferrl
