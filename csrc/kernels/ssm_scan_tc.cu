// Selective scan over whole sequences in chunks of 128 tokens on the 5th-generation tensor cores (models/mamba2.py); bf16
// inputs, float32 state.  With c_t the sum of the log decays up to token t of a chunk and S the state that enters it:
//
//   G = C B^T                                       [128 x 128]
//   Y = diag(2^c) C S + M X + D X,  M[t, s] = G[t, s] 2^(c_t - c_s) dt_s  for s <= t
//   S <- 2^c_last S + B^T X',       X'[s, :] = 2^(c_last - c_s) dt_s X[s, :]
//
// A CTA walks the chunks of one head and up to 64 of its columns.  The state never leaves tensor memory: it is the
// accumulator of B^T X', decayed in place between chunks.  M replaces G in tensor memory and is the A operand of M X.  B, C
// and X are used as TMA wrote them, K-major or MN-major as each product wants.
//
// Operands that are float32 by nature enter the products as sums of bf16 terms: X' as three (24 bits), so the state is as
// accurate as float32 multiplication makes it; M and the copy of S that feeds the outputs as two (16 bits), ahead of an
// output that is rounded to 8.
//
// 128 threads, thread = token = tensor-memory lane = state row; phases are separated by block barriers, and two CTAs on
// an SM fill each other's waits.  Every mbarrier wait is bounded and reports through the status word.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../api.h"
#include "../common.cuh"
#include "../gemm/tc_common.cuh"

namespace ferrl {
namespace {

using namespace tc;
using bf16 = __nv_bfloat16;

constexpr int kQ = 128;                          // tokens per chunk
constexpr int kAtom = kQ * 128;                  // [128 rows x 64 columns] bf16: 16 KB
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kAMajorMN = 1u << 15, kBMajorMN = 1u << 16;

// shared memory: C (2 atoms; the lowest term of X' later), B (2 atoms), X, S as two terms (the upper terms of X' later)
constexpr int kOffB = 2 * kAtom, kOffX = 4 * kAtom, kOffS = 5 * kAtom, kOffVec = 7 * kAtom;
constexpr int kSmem = kOffVec + kQ * 4 + 4 * 4 + 5 * 8 + 16;
static_assert(2 * (kSmem + 1024) <= 228 * 1024, "two CTAs per SM");

__device__ __forceinline__ uint32_t pair(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
__device__ __forceinline__ float2 unpair(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&v)); }
// byte offset of a row's 16-byte chunk in a 128B-swizzled [rows x 64 columns] tile
__device__ __forceinline__ int chunk_at(int row, int ch) { return row * 128 + ((ch ^ (row & 7)) << 4); }

__global__ void __launch_bounds__(kQ, 2)
ssm_scan_tc_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ CUtensorMap tmB, const __grid_constant__ CUtensorMap tmC,
                   SsmScanArgs a, int* status) {
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* sC = smem;
  uint8_t* sB = smem + kOffB;
  uint8_t* sX = smem + kOffX;
  uint8_t* sS = smem + kOffS;
  float* s_vec = reinterpret_cast<float*>(smem + kOffVec);       // log decay from s to the end of its 32 tokens + log2 dt_s
  float* s_sum = s_vec + kQ;                                     // log decay of each warp's tokens
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_sum + 4);
  uint64_t *full = bars, *g_done = bars + 1, *s_done = bars + 2, *y_done = bars + 3, *u_done = bars + 4;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 5);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int r = threadIdx.x, warp = r >> 5, lane = r & 31;
  const int p0 = blockIdx.x * 64, h = blockIdx.y, b = blockIdx.z, g = h / (a.H / a.G);
  const int n_atoms = (a.N + 63) / 64, k_steps = (a.N + 15) / 16;
  const int len = a.lens ? static_cast<int>(min(max(a.lens[b], 0ll), static_cast<long long>(a.T))) : a.T;
  const int chunks = (a.T + kQ - 1) / kQ;

  if (r == 0) {
    for (int i = 0; i < 5; ++i) mbar_init(&bars[i], 1);
    *abort_flag = (smem_u32(smem) & 1023) ? 1 : 0;
    if (*abort_flag) atomicCAS(status, kStatusOk, kStatusBadShape);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(256) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (n_atoms == 1) {                            // B^T X' always has 128 rows: the missing half of B is zero
    for (int i = r; i < kAtom / 16; i += kQ) reinterpret_cast<uint4*>(sB + kAtom)[i] = make_uint4(0, 0, 0, 0);
    fence_async_smem();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tG = tmem_base, tY = tmem_base + 128, tS = tmem_base + 192;
  const uint32_t lane_sel = static_cast<uint32_t>(warp * 32) << 16;

  auto load = [&](int c) {
    mbar_expect_tx(full, (2 * n_atoms + 1) * kAtom);
    for (int x = 0; x < n_atoms; ++x) {
      tma_load_4d(sC + x * kAtom, &tmC, full, x * 64, g, c * kQ, b);
      tma_load_4d(sB + x * kAtom, &tmB, full, x * 64, g, c * kQ, b);
    }
    tma_load_4d(sX, &tmX, full, p0, h, c * kQ, b);
  };
  const bf16* DT = static_cast<const bf16*>(a.dt) + b * a.dt_bs + h;
  auto step_of = [&](int c) {                    // raw step size of this thread's token; only those that count
    const int t = c * kQ + r;
    return t < len ? __bfloat162float(DT[t * a.dt_ts]) : -INFINITY;
  };
  const float A2 = -__expf(a.A_log[h]) * kLog2e, D = a.D[h], dtb = a.dt_bias[h];
  bf16* Y = static_cast<bf16*>(a.y) + static_cast<long long>(b) * a.T * a.H * a.P + static_cast<long long>(h) * a.P + p0;
  const int cols = min(64, a.P - p0);
  const uint64_t dC = make_smem_desc(smem_u32(sC)), dBk = make_smem_desc(smem_u32(sB));
  const uint64_t dBm = make_smem_desc_mn(smem_u32(sB), kAtom), dX = make_smem_desc_mn(smem_u32(sX), kAtom);
  const uint64_t dS = make_smem_desc_mn(smem_u32(sS), kAtom), dLow = make_smem_desc_mn(smem_u32(sC), kAtom);
  constexpr uint32_t id_g = make_idesc_bf16(128, 128), id_s = make_idesc_bf16(128, 64) | kBMajorMN,
                     id_u = make_idesc_bf16(128, 64) | kAMajorMN | kBMajorMN;

  bool ok = *abort_flag == 0;
  if (ok && r == 0) load(0);
  float raw = step_of(0);
  for (int c = 0; c < chunks && ok; ++c) {
    const uint32_t ph = c & 1;
    // ---- step sizes and log decays of the chunk
    const float z = raw + dtb;
    const float dt = raw == -INFINITY ? 0.f : (z > 20.f ? z : log1pf(__expf(z)));
    // sums over this warp's 32 tokens: up to and with this one, and behind it; every exponent below is a sum of terms of
    // one sign, so that a chunk's large total decay costs no accuracy between neighbours
    float loc = A2 * dt, suf = __shfl_down_sync(0xffffffffu, loc, 1);
    if (lane == 31) suf = 0.f;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float u = __shfl_up_sync(0xffffffffu, loc, o), d = __shfl_down_sync(0xffffffffu, suf, o);
      if (lane >= o) loc += u;
      if (lane + o < 32) suf += d;
    }
    if (lane == 31) s_sum[warp] = loc;
    __syncthreads();
    float before = 0.f, after = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float v = s_sum[w];
      if (w < warp) before += v;
      if (w > warp) after += v;
    }
    const float last = (s_sum[0] + s_sum[1]) + (s_sum[2] + s_sum[3]);
    s_vec[r] = suf + log2f(dt);                  // -inf where the token does not count
    // ---- the state that enters: two bf16 terms for C S, and its decayed self as the accumulator of B^T X'
    if (c > 0) {
      const float dec = exp2f(last);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t v[32], hi[16], lo[16];
        tmem_ld32(tS + lane_sel + half * 32, v);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const float x = __uint_as_float(v[2 * e]), y = __uint_as_float(v[2 * e + 1]);
          hi[e] = pair(x, y);
          const float2 f = unpair(hi[e]);
          lo[e] = pair(x - f.x, y - f.y);
          v[2 * e] = __float_as_uint(x * dec);
          v[2 * e + 1] = __float_as_uint(y * dec);
        }
        tmem_st32(tS + lane_sel + half * 32, v);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int at = chunk_at(r, half * 4 + k);
          *reinterpret_cast<uint4*>(sS + at) = make_uint4(hi[4 * k], hi[4 * k + 1], hi[4 * k + 2], hi[4 * k + 3]);
          *reinterpret_cast<uint4*>(sS + kAtom + at) = make_uint4(lo[4 * k], lo[4 * k + 1], lo[4 * k + 2], lo[4 * k + 3]);
        }
      }
      tmem_st_wait();
      fence_async_smem();
    }
    tc_fence_before();
    ok = mbar_wait(full, ph, abort_flag, status, kStatusWaitTimeoutProducer);
    if (__syncthreads_or(!ok)) { ok = false; break; }
    tc_fence_after();
    if (warp == 0) {
      if (elect_one()) {
        for (int k = 0; k < k_steps; ++k)
          umma(tG, desc_adv(dC, (k >> 2) * kAtom + (k & 3) * 32), desc_adv(dBk, (k >> 2) * kAtom + (k & 3) * 32), id_g, k > 0 ? 1u : 0u);
        umma_commit(g_done);
        if (c > 0) {
          for (int k = 0; k < 2 * k_steps; ++k) {
            const int term = k >= k_steps, kk = k - term * k_steps;
            umma(tY, desc_adv(dC, (kk >> 2) * kAtom + (kk & 3) * 32), desc_adv(dS, term * kAtom + kk * 2048), id_s, k > 0 ? 1u : 0u);
          }
          umma_commit(s_done);
        }
      }
      __syncwarp();
    }
    if (c + 1 < chunks) raw = step_of(c + 1);
    // ---- M in place of G: per 32 tokens s, 16 columns of upper terms, then 16 of lower ones
    ok = mbar_wait(g_done, ph, abort_flag, status, kStatusWaitTimeoutMma);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    if (ok) {
#pragma unroll 1
      for (int j = 0; j < 4; ++j) {
        uint32_t v[32], m[32];
        if (j <= warp) {
          tmem_ld32(tG + lane_sel + j * 32, v);
          tmem_ld_wait();
          if (j < warp) {
            float off = loc;                     // from the end of block j to this token
            for (int w = j + 1; w < warp; ++w) off += s_sum[w];
#pragma unroll
            for (int e = 0; e < 16; ++e) {
              const float2 bs = *reinterpret_cast<const float2*>(s_vec + j * 32 + 2 * e);
              v[2 * e] = __float_as_uint(__uint_as_float(v[2 * e]) * exp2f(off + bs.x));
              v[2 * e + 1] = __float_as_uint(__uint_as_float(v[2 * e + 1]) * exp2f(off + bs.y));
            }
          } else {                               // the diagonal block: the tokens are this warp's own
#pragma unroll
            for (int e = 0; e < 32; ++e) {
              const float f = exp2f(loc - __shfl_sync(0xffffffffu, loc, e)) * __shfl_sync(0xffffffffu, dt, e);
              v[e] = e > lane ? 0u : __float_as_uint(__uint_as_float(v[e]) * f);
            }
          }
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const float x = __uint_as_float(v[2 * e]), y = __uint_as_float(v[2 * e + 1]);
            m[e] = pair(x, y);
            const float2 f = unpair(m[e]);
            m[16 + e] = pair(x - f.x, y - f.y);
          }
        } else {
#pragma unroll
          for (int e = 0; e < 32; ++e) m[e] = 0u;
        }
        tmem_st32(tG + lane_sel + j * 32, m);
      }
      tmem_st_wait();
    }
    // ---- what the entering state gives every token
    if (c > 0) {
      ok = mbar_wait(s_done, (c - 1) & 1, abort_flag, status, kStatusWaitTimeoutMma) && ok;
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      if (ok) {
        const float f = exp2f(before + loc);
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t v[32];
          tmem_ld32(tY + lane_sel + half * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; ++e) v[e] = __float_as_uint(__uint_as_float(v[e]) * f);
          tmem_st32(tY + lane_sel + half * 32, v);
        }
        tmem_st_wait();
      }
    }
    // G and C S have retired for every warp before C and S are overwritten
    if (__syncthreads_or(!ok)) { ok = false; break; }
    {
      const float w = exp2f(suf + after) * dt;
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int at = chunk_at(r, k);
        const uint4 xv = *reinterpret_cast<const uint4*>(sX + at);
        const uint32_t xs[4] = {xv.x, xv.y, xv.z, xv.w};
        uint32_t t1[4], t2[4], t3[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = unpair(xs[e]);
          float x = f.x * w, y = f.y * w;
          t1[e] = pair(x, y);
          float2 q = unpair(t1[e]);
          x -= q.x;
          y -= q.y;
          t2[e] = pair(x, y);
          q = unpair(t2[e]);
          t3[e] = pair(x - q.x, y - q.y);
        }
        *reinterpret_cast<uint4*>(sS + at) = make_uint4(t1[0], t1[1], t1[2], t1[3]);
        *reinterpret_cast<uint4*>(sS + kAtom + at) = make_uint4(t2[0], t2[1], t2[2], t2[3]);
        *reinterpret_cast<uint4*>(sC + at) = make_uint4(t3[0], t3[1], t3[2], t3[3]);
      }
      fence_async_smem();
      tc_fence_before();
    }
    __syncthreads();
    tc_fence_after();
    if (warp == 0) {
      if (elect_one()) {
#pragma unroll
        for (int k = 0; k < 16; ++k) {           // upper terms, then lower ones
          const int kk = k & 7;
          umma_ts(tY, tG + (kk >> 1) * 32 + (kk & 1) * 8 + (k >> 3) * 16, desc_adv(dX, kk * 2048), id_s, (c > 0 || k > 0) ? 1u : 0u);
        }
        umma_commit(y_done);
#pragma unroll
        for (int k = 0; k < 24; ++k) {
          const int kk = k & 7;
          const uint64_t db = k < 16 ? desc_adv(dS, (k >> 3) * kAtom + kk * 2048) : desc_adv(dLow, kk * 2048);
          umma(tS, desc_adv(dBm, kk * 2048), db, id_u, (c > 0 || k > 0) ? 1u : 0u);
        }
        umma_commit(u_done);
      }
      __syncwarp();
    }
    // ---- outputs
    ok = mbar_wait(y_done, ph, abort_flag, status, kStatusWaitTimeoutEpilogue);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    if (ok) {
      const int t = c * kQ + r;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t v[32];
        tmem_ld32(tY + lane_sel + half * 32, v);
        tmem_ld_wait();
        if (t < a.T) {
          bf16* out = Y + static_cast<long long>(t) * a.H * a.P + half * 32;
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            if (half * 32 + k * 8 >= cols) break;
            const uint4 xv = *reinterpret_cast<const uint4*>(sX + chunk_at(r, half * 4 + k));
            const uint32_t xs[4] = {xv.x, xv.y, xv.z, xv.w};
            uint32_t o[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 f = unpair(xs[e]);
              o[e] = pair(__uint_as_float(v[k * 8 + 2 * e]) + D * f.x, __uint_as_float(v[k * 8 + 2 * e + 1]) + D * f.y);
            }
            *reinterpret_cast<uint4*>(out + k * 8) = make_uint4(o[0], o[1], o[2], o[3]);
          }
        }
        __syncwarp();
      }
      tc_fence_before();
    }
    // B and X' have been read and X is no longer needed: the next chunk may land
    ok = mbar_wait(u_done, ph, abort_flag, status, kStatusWaitTimeoutEpilogue) && ok;
    if (__syncthreads_or(!ok)) { ok = false; break; }
    tc_fence_after();
    if (r == 0 && c + 1 < chunks) load(c + 1);
  }
  if (ok && a.state) {
    float* So = a.state + ((static_cast<long long>(b) * a.H + h) * a.N + r) * a.P + p0;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      uint32_t v[32];
      tmem_ld32(tS + lane_sel + half * 32, v);
      tmem_ld_wait();
      if (r < a.N) {
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          if (half * 32 + k * 4 >= cols) break;
          *reinterpret_cast<uint4*>(So + half * 32 + k * 4) = make_uint4(v[4 * k], v[4 * k + 1], v[4 * k + 2], v[4 * k + 3]);
        }
      }
      __syncwarp();
    }
  }
  if (*abort_flag) {
    for (int i = 0; i < 64; ++i) __nanosleep(10000);   // let copies in flight land before shared memory goes away
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(256) : "memory");
  }
}

}  // namespace

bool ssm_scan_tc_supported(const SsmScanArgs& a) {
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return a.dtype == kBF16 && a.T >= 1 && a.N % 8 == 0 && a.N <= 128 && a.P % 8 == 0 && a.ts % 8 == 0 && a.bs % 8 == 0 && al16(a.x) && al16(a.Bm) &&
         al16(a.Cm) && al16(a.y) && al16(a.state);
}

const char* ssm_scan_tc(const SsmScanArgs& a, int* status, cudaStream_t s) {
  if (!ssm_scan_tc_supported(a)) return "ssm_scan_tc: unsupported arguments";
  if (a.B == 0) return nullptr;
  CUtensorMap tmX, tmB, tmC;
  if (!make_map_4d(&tmX, a.x, a.B, a.T, a.H, a.P, a.P, a.ts, a.bs, kQ) || !make_map_4d(&tmB, a.Bm, a.B, a.T, a.G, a.N, a.N, a.ts, a.bs, kQ) ||
      !make_map_4d(&tmC, a.Cm, a.B, a.T, a.G, a.N, a.N, a.ts, a.bs, kQ))
    return "ssm_scan_tc: tensor map failed";
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(ssm_scan_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem) == cudaSuccess &&
                             cudaFuncSetAttribute(ssm_scan_tc_kernel, cudaFuncAttributePreferredSharedMemoryCarveout, 100) == cudaSuccess))
    return "ssm_scan_tc: cannot reserve shared memory";
  ssm_scan_tc_kernel<<<dim3((a.P + 63) / 64, a.H, a.B), kQ, kSmem, s>>>(tmX, tmB, tmC, a, status);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "ssm_scan_tc launch failed";
}

}  // namespace ferrl
