// Residual sum, layer norm and depth average of a post-norm layer on a float32 stream, in one kernel:
//
//   t    = alpha * x + y * sigmoid(gate + gate_bias)        (y absent: t = x; gate absent: y as it is)
//   r    = (t - mean) / sqrt(mean((t - mean)^2) + eps) * w + b
//   next = sum_j coef[j] * history[j] + coef[n_hist] * r    (no coefficients: next = r)
//
// One CTA per row; t stays in shared memory between the passes.  Writes r and next (float32) and a copy of next in
// the compute dtype for the projections that follow.
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

template <typename TY, typename TG, typename TC, int V>
__global__ void post_norm_kernel(PostNormArgs a) {
  extern __shared__ __align__(16) float sm_t[];
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const long long row = blockIdx.x;
  const float* x = a.x + row * a.W;
  const TY* y = a.y ? static_cast<const TY*>(a.y) + row * a.ld_y : nullptr;
  const TG* g = a.gate ? static_cast<const TG*>(a.gate) + row * a.ld_gate : nullptr;
  float sum = 0.f;
  for (int c = threadIdx.x * V; c < a.W; c += blockDim.x * V) {
    Vec<V> t = ld<V>(x + c);
    if (y) {
      const Vec<V> yv = ld<V>(y + c);
      if (g) {
        const Vec<V> gv = ld<V>(g + c);
        Vec<V> gb;
        if (a.gate_bias) gb = ld<V>(a.gate_bias + c);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const float z = a.gate_bias ? gv.v[e] + gb.v[e] : gv.v[e];
          t.v[e] = a.alpha * t.v[e] + yv.v[e] / (1.f + __expf(-z));
        }
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) t.v[e] = a.alpha * t.v[e] + yv.v[e];
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) sum += t.v[e];
    st<V>(sm_t + c, t);
  }
  const float mean = block_sum(sum, red) / static_cast<float>(a.W);
  float sq = 0.f;
  for (int c = threadIdx.x * V; c < a.W; c += blockDim.x * V) {
    const Vec<V> t = ld<V>(sm_t + c);
#pragma unroll
    for (int e = 0; e < V; ++e) sq += (t.v[e] - mean) * (t.v[e] - mean);
  }
  const float rstd = 1.f / sqrtf(block_sum(sq, red) / static_cast<float>(a.W) + a.eps);
  const float last = a.coef ? a.coef[a.n_hist] : 1.f;
  for (int c = threadIdx.x * V; c < a.W; c += blockDim.x * V) {
    Vec<V> t = ld<V>(sm_t + c);
    const Vec<V> w = ld<V>(a.w + c);
    Vec<V> b;
    if (a.b) b = ld<V>(a.b + c);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      t.v[e] = (t.v[e] - mean) * rstd * w.v[e];
      if (a.b) t.v[e] += b.v[e];
    }
    if (a.r) st<V>(a.r + row * a.W + c, t);
    if (a.coef) {
#pragma unroll
      for (int e = 0; e < V; ++e) t.v[e] *= last;
      const float* hp = a.history + row * a.W + c;
#pragma unroll 4
      for (int j = 0; j < a.n_hist; ++j) {
        const Vec<V> h = ld<V>(hp + j * a.hist_stride);
        const float k = a.coef[j];
#pragma unroll
        for (int e = 0; e < V; ++e) t.v[e] += k * h.v[e];
      }
    }
    if (a.next) st<V>(a.next + row * a.W + c, t);
    if (a.cast) st<V>(static_cast<TC*>(a.cast) + row * a.W + c, t);
  }
}

template <typename TY, typename TG, typename TC>
const char* launch(const PostNormArgs& a, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(a.W) * 4;
  if (smem > 200 * 1024) return "post_norm: row too wide";
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = a.W % 4 == 0 && a.ld_y % 4 == 0 && a.ld_gate % 4 == 0 && a.hist_stride % 4 == 0 && al16(a.x) && al16(a.y) &&
                   (reinterpret_cast<uintptr_t>(a.gate) & (sizeof(TG) * 4 - 1)) == 0 && al16(a.gate_bias) && al16(a.w) && al16(a.b) &&
                   al16(a.history) && al16(a.r) && al16(a.next) && al16(a.cast);
  const int per = vec ? 4 : 1;
  const int threads = std::min(a.rows >= 1024 ? 256 : 1024, std::max(64, (a.W / per + 31) / 32 * 32));
  auto k4 = post_norm_kernel<TY, TG, TC, 4>;
  auto k1 = post_norm_kernel<TY, TG, TC, 1>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(k4, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess &&
                             cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess))
    return "post_norm: cannot reserve shared memory";
  launch_pdl(vec ? k4 : k1, dim3(static_cast<unsigned>(a.rows)), dim3(threads), smem, s, a);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "post_norm launch failed";
}

}  // namespace

const char* post_norm(const PostNormArgs& a, cudaStream_t s) {
  if (a.rows == 0) return nullptr;
  if (a.cast_dtype == kF32 && a.y_dtype == kF32 && a.gate_dtype == kF32) return launch<float, float, float>(a, s);
  if (a.cast_dtype == kBF16 && a.y_dtype == kBF16 && a.gate_dtype == kBF16) return launch<bf16, bf16, bf16>(a, s);
  if (a.cast_dtype == kBF16 && a.y_dtype == kBF16 && a.gate_dtype == kF32) return launch<bf16, float, bf16>(a, s);
  return "post_norm: unsupported dtype combination";
}

}  // namespace ferrl
