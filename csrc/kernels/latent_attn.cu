// Latent attention (models/latent.py): keys and values of all heads come from one low-rank latent per token.
//
//   latent_prep_kernel      RMS norm of the latent, rotation of the shared key part and of the queries; writes the
//                           row [latent | rotated key part] to a packed buffer or to its slot of a ring cache
//   latent_fwd_any_kernel   causal (windowed) attention over whole sequences, any sizes, bf16 or fp32
//                           (flash_tc.cu holds the tcgen05 form for bf16)
//   head_gemm_kernel        out[b, h, :] = W[h] x[b, h, :], one small matrix per head (query absorption, value
//                           expansion of a decode step) on mma.sync; head_gemm_any_kernel for other types and sizes
//   latent_decode_any_kernel  one query per row against the row's cached latents, any type and size
//                           (latent_decode_tc.cu holds the tcgen05 form for bf16); attn_combine_kernel joins key ranges
//
// Scores, softmax and sink are fp32.  A sink adds exp(sink_h) to the softmax denominator of head h.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <algorithm>

#include "../api.h"
#include "../common.cuh"
#include "mma_sync.cuh"

namespace ferrl {
namespace {

using bf16 = __nv_bfloat16;
constexpr float kLog2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------------ prep / append
template <typename T>
__global__ void latent_prep_kernel(LatentPrepArgs a) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[32];
  const long long t = blockIdx.x;
  long long pos = a.kv_len ? a.kv_len[t] : a.pos[t % a.S];
  const long long slot = pos;
  pos = min(max(pos, 0ll), a.max_pos - 1);
  const float* cs = a.cos_t + pos * a.half;
  const float* sn = a.sin_t + pos * a.half;
  const T* d = static_cast<const T*>(a.dkv) + t * a.ld_dkv;
  T* row = static_cast<T*>(a.out) + (a.kv_len ? (t * a.slots + slot % a.slots) : t) * a.width;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.rank; i += blockDim.x) {
    const float v = to_f(d[i]);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / static_cast<float>(a.rank) + a.eps);
  for (int i = threadIdx.x; i < a.rank; i += blockDim.x) row[i] = from_f<T>(to_f(d[i]) * r * a.norm_w[i]);
  // rotated key part: pairs (i, i + half); entries past 2 * half pass through
  for (int i = threadIdx.x; i < a.half; i += blockDim.x) {
    const float u = to_f(d[a.rank + i]), v = to_f(d[a.rank + a.half + i]);
    row[a.rank + i] = from_f<T>(u * cs[i] - v * sn[i]);
    row[a.rank + a.half + i] = from_f<T>(v * cs[i] + u * sn[i]);
  }
  for (int i = 2 * a.half + threadIdx.x; i < a.rot; i += blockDim.x) row[a.rank + i] = d[a.rank + i];
  for (int i = a.rank + a.rot + threadIdx.x; i < a.width; i += blockDim.x) row[i] = from_f<T>(0.f);
  T* q = static_cast<T*>(a.q) + t * a.ld_q;
  const int E = a.dim + a.rot;
  for (int i = threadIdx.x; i < a.heads * a.half; i += blockDim.x) {
    const int h = i / a.half, p = i - h * a.half;
    T* x = q + static_cast<long long>(h) * E + a.dim + p;
    const float u = to_f(x[0]), v = to_f(x[a.half]);
    x[0] = from_f<T>(u * cs[p] - v * sn[p]);
    x[a.half] = from_f<T>(v * cs[p] + u * sn[p]);
  }
}

// ------------------------------------------------------------------------------------------------ prefill, any sizes
constexpr int kAnyQ = 16, kAnyK = 32;

template <typename T>
__global__ void __launch_bounds__(128) latent_fwd_any_kernel(LatentFwdArgs a) {
  extern __shared__ float sm[];
  const int E = a.dim + a.rot, KS = E + 1;
  float* sk = sm;                          // [kAnyK][E + 1]
  float* sv = sk + kAnyK * KS;             // [kAnyK][vdim]
  float* sq = sv + kAnyK * a.vdim;         // [kAnyQ][E]
  float* so = sq + kAnyQ * E;              // [kAnyQ][vdim]
  float* sp = so + kAnyQ * a.vdim;         // [4 warps][kAnyK]
  const int h = blockIdx.y, b = blockIdx.z, q0 = blockIdx.x * kAnyQ;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* Q = static_cast<const T*>(a.q) + b * a.q_bs + static_cast<long long>(h) * E;
  const T* KN = static_cast<const T*>(a.kn) + b * a.kn_bs + static_cast<long long>(h) * a.dim;
  const T* KR = static_cast<const T*>(a.kr) + b * a.kr_bs;
  const T* V = static_cast<const T*>(a.v) + b * a.v_bs + static_cast<long long>(h) * a.vdim;
  for (int i = threadIdx.x; i < kAnyQ * E; i += 128) {
    const int r = i / E, c = i - r * E;
    sq[i] = q0 + r < a.S ? to_f(Q[(q0 + r) * a.q_ts + c]) : 0.f;
  }
  for (int i = threadIdx.x; i < kAnyQ * a.vdim; i += 128) so[i] = 0.f;
  float m[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) { m[i] = -INFINITY; l[i] = 0.f; }
  const int last = min(q0 + kAnyQ, a.S) - 1;
  const int j_lo = a.window > 0 ? max(0, q0 - a.window + 1) / kAnyK * kAnyK : 0;
  for (int j0 = j_lo; j0 <= last; j0 += kAnyK) {
    __syncthreads();
    for (int i = threadIdx.x; i < kAnyK * E; i += 128) {
      const int r = i / E, c = i - r * E;
      float v = 0.f;
      if (j0 + r < a.S) v = c < a.dim ? to_f(KN[(j0 + r) * a.kn_ts + c]) : to_f(KR[(j0 + r) * a.kr_ts + c - a.dim]);
      sk[r * KS + c] = v;
    }
    for (int i = threadIdx.x; i < kAnyK * a.vdim; i += 128) {
      const int r = i / a.vdim, c = i - r * a.vdim;
      sv[i] = j0 + r < a.S ? to_f(V[(j0 + r) * a.v_ts + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int qi = 0; qi < 4; ++qi) {
      const int r = warp * 4 + qi, pos = q0 + r, key = j0 + lane;
      float s = -INFINITY;
      if (key <= pos && pos < a.S && (a.window <= 0 || pos - key < a.window)) {
        s = 0.f;
        for (int c = 0; c < E; ++c) s += sq[r * E + c] * sk[lane * KS + c];
        s *= a.scale;
      }
      const float mn = fmaxf(m[qi], warp_max(s));
      if (mn == -INFINITY) continue;       // warp-uniform: nothing visible yet
      const float p = s == -INFINITY ? 0.f : exp2f((s - mn) * kLog2e);
      const float corr = m[qi] == -INFINITY ? 0.f : exp2f((m[qi] - mn) * kLog2e);
      l[qi] = l[qi] * corr + warp_sum(p);
      m[qi] = mn;
      sp[warp * kAnyK + lane] = p;
      __syncwarp();
      for (int c = lane; c < a.vdim; c += 32) {
        float o = so[r * a.vdim + c] * corr;
        for (int k = 0; k < kAnyK; ++k) o += sp[warp * kAnyK + k] * sv[k * a.vdim + c];
        so[r * a.vdim + c] = o;
      }
      __syncwarp();
    }
  }
#pragma unroll
  for (int qi = 0; qi < 4; ++qi) {
    const int r = warp * 4 + qi, pos = q0 + r;
    if (pos >= a.S) continue;
    float den = l[qi];
    if (a.sink) den += exp2f((a.sink[h] - m[qi]) * kLog2e);
    const float inv = 1.f / den;
    T* o = static_cast<T*>(a.out) + b * a.o_bs + pos * a.o_ts + static_cast<long long>(h) * a.vdim;
    for (int c = lane; c < a.vdim; c += 32) o[c] = from_f<T>(so[r * a.vdim + c] * inv);
  }
}

// ------------------------------------------------------------------------------------------------ per-head matrices
template <typename T>
__global__ void head_gemm_any_kernel(const T* __restrict__ x, long long ldx, int xh, const T* __restrict__ w,
                                     T* __restrict__ out, long long ldo, int B, int N, int K) {
  const int h = blockIdx.y, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* xr = x + b * ldx + static_cast<long long>(h) * xh;
  for (int n = blockIdx.x * 8 + warp; n < N; n += gridDim.x * 8) {
    const T* wr = w + (static_cast<long long>(h) * N + n) * K;
    float s = 0.f;
    for (int k = lane; k < K; k += 32) s += to_f(xr[k]) * to_f(wr[k]);
    s = warp_sum(s);
    if (lane == 0) out[b * ldo + static_cast<long long>(h) * N + n] = from_f<T>(s);
  }
}

// 64 rows x 64 columns per CTA, k in steps of 64 through a DEPTH-stage cp.async ring; K % 8 == 0.  The matrices are
// weights, so the first stages of w are requested before the wait for the predecessor that writes x.
constexpr int kHgStage = 2 * 64 * 128;     // bytes: x tile + w tile
template <int DEPTH>
__global__ void __launch_bounds__(128) head_gemm_kernel(const bf16* __restrict__ x, long long ldx, int xh,
                                                        const bf16* __restrict__ w, bf16* __restrict__ out,
                                                        long long ldo, int B, int N, int K) {
  using namespace mmah;
  pdl_trigger();
  extern __shared__ __align__(1024) uint8_t hg_smem[];
  const int n0 = blockIdx.x * 64, b0 = blockIdx.y * 64, h = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wm = warp & 1, wn = warp >> 1;
  const bf16* xb = x + static_cast<long long>(h) * xh;
  const bf16* wb = w + static_cast<long long>(h) * N * K;
  const uint32_t base = smem_addr(hg_smem);
  const int nk = (K + 63) / 64;
  auto load_w = [&](int kt) {
    if (kt >= nk) return;
    const uint32_t s = base + (kt % DEPTH) * kHgStage + 64 * 128;
    for (int i = threadIdx.x; i < 64 * 8; i += 128) {
      const int r = i >> 3, c = i & 7, k = kt * 64 + c * 8;
      const bool ok = n0 + r < N && k < K;
      cp_async16(s + sw_off<128>(r, c), ok ? wb + static_cast<long long>(n0 + r) * K + k : wb, ok);
    }
  };
  auto load_x = [&](int kt) {               // closes the stage's copy group (an empty one past the end)
    const uint32_t s = base + (kt % DEPTH) * kHgStage;
    for (int i = threadIdx.x; kt < nk && i < 64 * 8; i += 128) {
      const int r = i >> 3, c = i & 7, k = kt * 64 + c * 8;
      const bool ok = b0 + r < B && k < K;
      cp_async16(s + sw_off<128>(r, c), ok ? xb + (b0 + r) * ldx + k : xb, ok);
    }
    cp_commit();
  };
#pragma unroll
  for (int kt = 0; kt < DEPTH - 1; ++kt) load_w(kt);
  pdl_wait();
#pragma unroll
  for (int kt = 0; kt < DEPTH - 1; ++kt) load_x(kt);
  float acc[2][4][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  for (int kt = 0; kt < nk; ++kt) {
    cp_wait<DEPTH - 2>();                 // one group a stage, empty ones included: stage kt has landed
    __syncthreads();                         // and everyone is done with the stage that is loaded next
    load_w(kt + DEPTH - 1);
    load_x(kt + DEPTH - 1);
    const uint32_t s = base + (kt % DEPTH) * kHgStage;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t a[2][4], bb[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
        ldsm4(s + sw_off<128>(wm * 32 + i * 16 + (lane & 15), ks * 2 + (lane >> 4)), a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
      for (int j = 0; j < 2; ++j)      // 16 columns: {n 0-7 k 0-7, n 0-7 k 8-15, n 8-15 k 0-7, n 8-15 k 8-15}
        ldsm4(s + 64 * 128 + sw_off<128>(wn * 32 + j * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1)),
              bb[j][0], bb[j][1], bb[j][2], bb[j][3]);
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) mma16816(acc[i][j], a[i], bb[j >> 1][(j & 1) * 2], bb[j >> 1][(j & 1) * 2 + 1]);
    }
  }
  cp_wait<0>();
  bf16* ob = out + static_cast<long long>(h) * N;
  const bool pairs = (N % 2) == 0 && (ldo % 2) == 0;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int r = b0 + wm * 32 + i * 16 + (lane >> 2) + (e >> 1) * 8;
        const int c = n0 + wn * 32 + j * 8 + (lane & 3) * 2;
        if (r >= B || c >= N) continue;
        if (pairs) {
          *reinterpret_cast<uint32_t*>(ob + r * ldo + c) = pack_bf16(acc[i][j][e], acc[i][j][e + 1]);
        } else {
          ob[r * ldo + c] = __float2bfloat16_rn(acc[i][j][e]);
          if (c + 1 < N) ob[r * ldo + c + 1] = __float2bfloat16_rn(acc[i][j][e + 1]);
        }
      }
}

// ------------------------------------------------------------------------------------------------ decode, any sizes
template <typename T>
__global__ void __launch_bounds__(128) latent_decode_any_kernel(LatentDecodeArgs a) {
  extern __shared__ float sm[];
  float* sq = sm;                       // [rank + rot]
  float* so = sq + a.rank + a.rot;      // [rank]
  __shared__ float sp[128], red[32];
  const int h = blockIdx.x, b = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int E = a.rank + a.rot;
  const int n = min(max(a.count[b], 0), a.slots);
  const T* qa = static_cast<const T*>(a.qa) + (static_cast<long long>(b) * a.heads + h) * a.rank;
  const T* qr = static_cast<const T*>(a.qr) + b * a.ld_qr + static_cast<long long>(h) * a.qr_hs;
  const T* cache = static_cast<const T*>(a.cache) + static_cast<long long>(b) * a.slots * a.width;
  for (int i = threadIdx.x; i < E; i += 128) sq[i] = i < a.rank ? to_f(qa[i]) : to_f(qr[i - a.rank]);
  for (int i = threadIdx.x; i < a.rank; i += 128) so[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < n; k0 += 128) {
    const int nk = min(128, n - k0);
    __syncthreads();
    for (int k = warp; k < nk; k += 4) {
      const T* row = cache + static_cast<long long>(k0 + k) * a.width;
      float s = 0.f;
      for (int c = lane; c < E; c += 32) s += sq[c] * to_f(row[c]);
      s = warp_sum(s) * a.scale;
      if (lane == 0) sp[k] = s;
    }
    __syncthreads();
    float s = static_cast<int>(threadIdx.x) < nk ? sp[threadIdx.x] : -INFINITY;
    const float mn = fmaxf(m, block_max(s, red));
    const float p = s == -INFINITY ? 0.f : exp2f((s - mn) * kLog2e);
    const float corr = m == -INFINITY ? 0.f : exp2f((m - mn) * kLog2e);
    l = l * corr + block_sum(p, red);
    m = mn;
    sp[threadIdx.x] = p;
    __syncthreads();
    for (int c = threadIdx.x; c < a.rank; c += 128) {
      float o = so[c] * corr;
      for (int k = 0; k < nk; ++k) o += sp[k] * to_f(cache[static_cast<long long>(k0 + k) * a.width + c]);
      so[c] = o;
    }
  }
  float inv = 0.f;
  if (n > 0) inv = 1.f / (a.sink ? l + exp2f((a.sink[h] - m) * kLog2e) : l);
  __syncthreads();
  T* o = static_cast<T*>(a.ctx) + (static_cast<long long>(b) * a.heads + h) * a.rank;
  for (int c = threadIdx.x; c < a.rank; c += 128) o[c] = from_f<T>(so[c] * inv);
}

// ------------------------------------------------------------------------------------------------ key ranges of a row
__global__ void attn_combine_kernel(const float* __restrict__ ws, const float* __restrict__ sink, bf16* __restrict__ ctx,
                                      int heads, int rank, int n_splits) {
  pdl_trigger();
  pdl_wait();
  const long long oh = blockIdx.x;
  const float* p = ws + oh * n_splits * (rank + 2);
  float m = -INFINITY;
  for (int s = 0; s < n_splits; ++s) m = fmaxf(m, p[static_cast<long long>(s) * (rank + 2) + rank]);
  float l = 0.f;
  for (int s = 0; s < n_splits; ++s) {
    const float* q = p + static_cast<long long>(s) * (rank + 2) + rank;
    if (q[0] != -INFINITY) l += q[1] * exp2f(q[0] - m);
  }
  float inv = 0.f;
  if (m != -INFINITY) inv = 1.f / (sink ? l + exp2f(sink[oh % heads] * kLog2e - m) : l);
  for (int c = threadIdx.x; c < rank; c += blockDim.x) {
    float o = 0.f;
    for (int s = 0; s < n_splits; ++s) {
      const float* q = p + static_cast<long long>(s) * (rank + 2);
      if (q[rank] != -INFINITY) o += q[c] * exp2f(q[rank] - m);
    }
    ctx[oh * rank + c] = __float2bfloat16_rn(o * inv);
  }
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

const char* latent_prep(const LatentPrepArgs& a, cudaStream_t s) {
  if (a.n_tok == 0) return nullptr;
  const int threads = a.rank + a.heads * a.half > 512 ? 256 : 128;
  if (a.dtype == kF32) launch_pdl(latent_prep_kernel<float>, dim3(a.n_tok), dim3(threads), 0, s, a);
  else launch_pdl(latent_prep_kernel<bf16>, dim3(a.n_tok), dim3(threads), 0, s, a);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "latent_prep launch failed";
}

const char* latent_fwd_any(const LatentFwdArgs& a, cudaStream_t s) {
  if (a.B == 0 || a.S == 0) return nullptr;
  const int E = a.dim + a.rot;
  const size_t smem = (static_cast<size_t>(kAnyK) * (E + 1 + a.vdim) + kAnyQ * (E + a.vdim) + 4 * kAnyK) * 4;
  if (smem > 227 * 1024) return "latent_fwd: head sizes too large";
  const dim3 grid((a.S + kAnyQ - 1) / kAnyQ, a.heads, a.B);
  if (!FERRL_ONCE_PER_DEVICE(
          cudaFuncSetAttribute(latent_fwd_any_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) == cudaSuccess &&
          cudaFuncSetAttribute(latent_fwd_any_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) == cudaSuccess))
    return "latent_fwd: cannot reserve shared memory";
  if (a.dtype == kF32) latent_fwd_any_kernel<float><<<grid, 128, smem, s>>>(a);
  else latent_fwd_any_kernel<bf16><<<grid, 128, smem, s>>>(a);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "latent_fwd launch failed";
}

const char* head_gemm(int dtype, const void* x, long long ldx, int xh, const void* w, void* out, long long ldo, int B, int H,
                      int N, int K, cudaStream_t s) {
  if (B == 0) return nullptr;
  if (dtype == kBF16 && K % 8 == 0 && ldx % 8 == 0 && xh % 8 == 0 && al16(x) && al16(w)) {
    const bf16 *xp = static_cast<const bf16*>(x), *wp = static_cast<const bf16*>(w);
    const dim3 grid((N + 63) / 64, (B + 63) / 64, H);
    // short contractions take three stages (four CTAs an SM), long ones five
    if (!FERRL_ONCE_PER_DEVICE(
            cudaFuncSetAttribute(head_gemm_kernel<3>, cudaFuncAttributeMaxDynamicSharedMemorySize, 3 * kHgStage) == cudaSuccess &&
            cudaFuncSetAttribute(head_gemm_kernel<5>, cudaFuncAttributeMaxDynamicSharedMemorySize, 5 * kHgStage) == cudaSuccess))
      return "head_gemm: cannot reserve shared memory";
    if (K <= 128) launch_pdl(head_gemm_kernel<3>, grid, dim3(128), 3 * kHgStage, s, xp, ldx, xh, wp, static_cast<bf16*>(out), ldo, B, N, K);
    else launch_pdl(head_gemm_kernel<5>, grid, dim3(128), 5 * kHgStage, s, xp, ldx, xh, wp, static_cast<bf16*>(out), ldo, B, N, K);
  } else {
    const dim3 grid(std::min((N + 7) / 8, 64), H, B);
    if (dtype == kF32)
      head_gemm_any_kernel<float><<<grid, 256, 0, s>>>(static_cast<const float*>(x), ldx, xh, static_cast<const float*>(w),
                                                       static_cast<float*>(out), ldo, B, N, K);
    else
      head_gemm_any_kernel<bf16><<<grid, 256, 0, s>>>(static_cast<const bf16*>(x), ldx, xh, static_cast<const bf16*>(w),
                                                      static_cast<bf16*>(out), ldo, B, N, K);
  }
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "head_gemm launch failed";
}

const char* latent_decode(const LatentDecodeArgs& a, int n_splits, int* status, cudaStream_t s) {
  if (a.B == 0) return nullptr;
  if (!latent_decode_tc_supported(a)) {
    const size_t smem = static_cast<size_t>(2 * a.rank + a.rot) * 4;
    if (smem > 200 * 1024) return "latent_decode: latent too large";
    const dim3 grid(a.heads, a.B);
    if (!FERRL_ONCE_PER_DEVICE(
            cudaFuncSetAttribute(latent_decode_any_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess &&
            cudaFuncSetAttribute(latent_decode_any_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) == cudaSuccess))
      return "latent_decode: cannot reserve shared memory";
    if (a.dtype == kF32) latent_decode_any_kernel<float><<<grid, 128, smem, s>>>(a);
    else latent_decode_any_kernel<bf16><<<grid, 128, smem, s>>>(a);
    count_launch();
    return cudaGetLastError() == cudaSuccess ? nullptr : "latent_decode launch failed";
  }
  if (n_splits > 1 && !a.ws) return "latent_decode: workspace missing";
  if (const char* err = latent_decode_tc(a, n_splits, status, s)) return err;
  if (n_splits > 1) return attn_combine(a.ws, a.sink, a.ctx, static_cast<long long>(a.B) * a.heads, a.heads, a.rank, n_splits, s);
  return cudaGetLastError() == cudaSuccess ? nullptr : "latent_decode launch failed";
}

const char* attn_combine(const float* ws, const float* sink, void* out, long long heads_total, int heads, int width, int n_splits, cudaStream_t s) {
  launch_pdl(attn_combine_kernel, dim3(static_cast<unsigned>(heads_total)), dim3(128), 0, s, ws, sink, static_cast<bf16*>(out), heads, width, n_splits);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "attn_combine launch failed";
}

}  // namespace ferrl
