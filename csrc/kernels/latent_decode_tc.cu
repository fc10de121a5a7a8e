// One query per row against the row's cached latents, on the 5th-generation tensor cores (models/latent.py).
//
// The heads of a row share one pass over its cache.  A CTA owns NH heads of one row and a range of the cached tokens and
// works on tiles of 128 tokens in transposed form, so that the 128 rows of an MMA are always tokens or latent entries
// and never heads:
//
//   S^T [128 tokens x NH heads]   = C Q^T       C: the tile as TMA wrote it (K-major), Q: absorbed and rotated queries
//   O^T [128 latents x NH heads] += C^T P       C^T: the same bytes through an MN-major descriptor, one MMA block per 128
//                                               latent entries, accumulated in tensor memory over the tiles
//
//   warp 0      TMA producer: the queries once, then each tile as 64-column atoms (latent atoms, then the rotated part)
//   warp 1      tcgen05.mma issue; a latent block's atoms go back to the producer as soon as its O^T MMAs have retired
//   warps 2-5   softmax: a thread owns one token and all NH heads; maxima and sums over the tokens by a halving exchange
//               inside the warp (lane = head afterwards) and a small shared array between the warps; O^T is rescaled only
//               when a head's maximum grew by more than 2^8.  P goes to the shared memory of the tile's rotated atom,
//               which nothing reads any more.
//
// Every wait is bounded and reports through the status word.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <algorithm>

#include "../api.h"
#include "../common.cuh"
#include "../gemm/tc_common.cuh"

namespace ferrl {
namespace {

using namespace tc;
using bf16 = __nv_bfloat16;

constexpr int kTok = 128;                       // tokens per tile
constexpr int kAtom = kTok * 128;               // [128 tokens x 64 columns] bf16: 16 KB
constexpr int kMaxAtoms = 11;
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kAMajorMN = 1u << 15;        // instruction descriptor: A operand is MN-major

struct LatentTcGeom {
  int na_lat, na, stages, tmem_cols;            // latent atoms, all atoms of a row, tiles in shared memory
  unsigned long long kmask;                     // bit 4 * atom + step: that 16-column step is not all padding
  int* status;
};

// 32 values per lane, reduced over the lanes: lane l returns the result of value l (31 exchanges)
template <bool MAX>
__device__ __forceinline__ float halving_reduce(const float* in, int lane) {
  float v[32];
#pragma unroll
  for (int j = 0; j < 32; ++j) v[j] = in[j];
#pragma unroll
  for (int w = 16; w >= 1; w >>= 1) {
    const bool up = (lane & w) != 0;
#pragma unroll
    for (int j = 0; j < w; ++j) {
      const float send = up ? v[j] : v[j + w], keep = up ? v[j + w] : v[j];
      const float got = __shfl_xor_sync(0xffffffffu, send, w);
      v[j] = MAX ? fmaxf(keep, got) : keep + got;
    }
  }
  return v[0];
}

template <int NH>
__global__ void __launch_bounds__(192, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmCr,
                        const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmQr, LatentDecodeArgs a,
                        int n_splits, LatentTcGeom g) {
  constexpr int NG = NH / 32;                   // groups of 32 heads
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sC = sQ + g.na * (NH * 128);
  float* s_max = reinterpret_cast<float*>(sC + g.stages * g.na * kAtom);   // [2 tiles][4 warps][NH]
  float* s_vec = s_max + 2 * 4 * NH;            // [4 warps][NH] maxima in use, at the end 1 / denominator
  float* s_cor = s_vec + 4 * NH;                // [4 warps][NH] rescale factors, at the end the row sums
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_cor + 4 * NH);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;                  // [2]
  uint64_t* p_full = bars + 3;
  uint64_t* o_done = bars + 4;
  uint64_t* warps_in = bars + 5;                // the four softmax warps meet here once a tile and once at the end
  uint64_t* full = bars + 6;                    // [stages * na]
  uint64_t* empty = full + 2 * kMaxAtoms;       // [stages * na]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(empty + 2 * kMaxAtoms);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, hb = blockIdx.y * NH, b = blockIdx.z;
  const int n_blocks = (g.na_lat + 1) / 2;      // 128-entry blocks of the latent
  pdl_trigger();
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    mbar_init(p_full, 4);
    mbar_init(o_done, 1);
    mbar_init(warps_in, 4);
    for (int i = 0; i < g.stages * g.na; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(g.tmem_cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_wait();                                   // counts, queries and the newest cache rows come from the predecessors
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tO = tmem_base, tS = tmem_base + n_blocks * NH;           // S^T buffers at tS and tS + NH
  const int n = min(max(a.count[b], 0), a.slots);
  const int tiles = (n + kTok - 1) / kTok;
  const int t_lo = static_cast<int>(static_cast<long long>(tiles) * split / n_splits);
  const int n_t = static_cast<int>(static_cast<long long>(tiles) * (split + 1) / n_splits) - t_lo;

  if (warp == 0) {
    if (lane == 0 && n_t > 0) {
      // ------------------------------------------------------------------ TMA producer
      mbar_expect_tx(q_full, g.na * NH * 128);
      for (int x = 0; x < g.na; ++x) {
        if (x < g.na_lat) tma_load_3d(sQ + x * (NH * 128), &tmQ, q_full, x * 64, hb, b);
        else tma_load_3d(sQ + x * (NH * 128), &tmQr, q_full, (x - g.na_lat) * 64, hb, b);
      }
      bool ok = true;
      for (int i = 0; i < n_t && ok; ++i) {
        const int st = g.stages == 2 ? (i & 1) : 0, use = g.stages == 2 ? (i >> 1) : i;
        for (int x = 0; x < g.na; ++x) {
          const int s = st * g.na + x;
          if (use > 0 && !mbar_wait(&empty[s], (use - 1) & 1, abort_flag, g.status, kStatusWaitTimeoutProducer)) { ok = false; break; }
          mbar_expect_tx(&full[s], kAtom);
          if (x < g.na_lat) tma_load_3d(sC + s * kAtom, &tmC, &full[s], x * 64, (t_lo + i) * kTok, b);
          else tma_load_3d(sC + s * kAtom, &tmCr, &full[s], (x - g.na_lat) * 64, (t_lo + i) * kTok, b);
        }
      }
      if (*abort_flag) {
        for (int i = 0; i < 64; ++i) __nanosleep(10000);   // let copies in flight land before shared memory goes away
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA warp: all lanes walk the loop, one issues
    constexpr uint32_t idesc_s = make_idesc_bf16(128, NH), idesc_o = make_idesc_bf16(128, NH) | kAMajorMN;
    auto issue_s = [&](int i) -> bool {
      const int st = g.stages == 2 ? (i & 1) : 0, use = g.stages == 2 ? (i >> 1) : i;
      for (int x = 0; x < g.na; ++x) {
        const int s = st * g.na + x;
        if (!mbar_wait_warp(&full[s], use & 1, abort_flag, g.status, kStatusWaitTimeoutMma)) return false;
        tc_fence_after();
        const uint64_t dc = make_smem_desc(smem_u32(sC + s * kAtom)), dq = make_smem_desc(smem_u32(sQ + x * (NH * 128)));
        const uint32_t steps = static_cast<uint32_t>(g.kmask >> (4 * x)) & 15u;
        if (elect_one()) {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if ((steps >> k) & 1u)
              umma(tS + (i & 1) * NH, desc_adv(dc, k * 32), desc_adv(dq, k * 32), idesc_s, (x > 0 || k > 0) ? 1u : 0u);
          if (x == g.na - 1) umma_commit(&s_full[i & 1]);
        }
        __syncwarp();
      }
      return true;
    };
    auto issue_o = [&](int i) -> bool {
      const int st = g.stages == 2 ? (i & 1) : 0;
      if (!mbar_wait_warp(p_full, i & 1, abort_flag, g.status, kStatusWaitTimeoutMma)) return false;
      tc_fence_after();
      const uint64_t dp = make_smem_desc(smem_u32(sC + (st * g.na + g.na_lat) * kAtom));
      for (int m = 0; m < n_blocks; ++m) {
        const uint64_t dc = make_smem_desc_mn(smem_u32(sC + (st * g.na + 2 * m) * kAtom), kAtom);
        if (elect_one()) {
#pragma unroll
          for (int k = 0; k < kTok / 16; ++k)
            umma(tO + m * NH, desc_adv(dc, k * 2048), desc_adv(dp, (k >> 2) * (NH * 128) + (k & 3) * 32), idesc_o, (i > 0 || k > 0) ? 1u : 0u);
          umma_commit(&empty[st * g.na + 2 * m]);
          if (2 * m + 1 < g.na_lat) umma_commit(&empty[st * g.na + 2 * m + 1]);
          if (m == n_blocks - 1) {
            for (int x = g.na_lat; x < g.na; ++x) umma_commit(&empty[st * g.na + x]);
            umma_commit(o_done);
          }
        }
        __syncwarp();
      }
      return true;
    };
    bool ok = n_t > 0 && mbar_wait_warp(q_full, 0, abort_flag, g.status, kStatusWaitTimeoutMma);
    if (ok) ok = issue_s(0);
    for (int i = 0; i < n_t && ok; ++i) {
      // with two tiles in shared memory the next tile's scores are computed under this tile's softmax
      if (g.stages == 2 && i + 1 < n_t) ok = issue_s(i + 1);
      if (ok) ok = issue_o(i);
      if (ok && g.stages == 1 && i + 1 < n_t) ok = issue_s(i + 1);
    }
  } else {
    // ------------------------------------------------------------------ softmax and output
    const int q = warp & 3, r = q * 32 + lane;  // token inside the tile == tensor-memory lane
    const uint32_t lane_sel = static_cast<uint32_t>(q * 32) << 16;
    const float c2 = a.scale * kLog2e;
    float m_used[NG], l_run[NG];                // lane = head (of each group), the same in all four warps
#pragma unroll
    for (int v = 0; v < NG; ++v) { m_used[v] = -INFINITY; l_run[v] = 0.f; }
    float* my_vec = s_vec + q * NH;
    float* my_cor = s_cor + q * NH;
    bool ok = true;
    for (int i = 0; i < n_t; ++i) {
      if (!mbar_wait_warp(&s_full[i & 1], (i >> 1) & 1, abort_flag, g.status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
      tc_fence_after();
      float sv[NH];
#pragma unroll
      for (int v = 0; v < NG; ++v) tmem_ld32(tS + (i & 1) * NH + lane_sel + v * 32, reinterpret_cast<uint32_t*>(sv) + v * 32);
      tmem_ld_wait();
      const bool live = (t_lo + i) * kTok + r < n;
#pragma unroll
      for (int e = 0; e < NH; ++e) sv[e] = live ? sv[e] * c2 : -INFINITY;
      float* mx_buf = s_max + (i & 1) * 4 * NH;
#pragma unroll
      for (int v = 0; v < NG; ++v) mx_buf[q * NH + v * 32 + lane] = halving_reduce<true>(sv + v * 32, lane);
      __syncwarp();
      if (lane == 0) mbar_arrive(warps_in);
      if (!mbar_wait_warp(warps_in, i & 1, abort_flag, g.status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
      bool grew = false;
#pragma unroll
      for (int v = 0; v < NG; ++v) {
        const int h = v * 32 + lane;
        const float mx = fmaxf(fmaxf(mx_buf[h], mx_buf[NH + h]), fmaxf(mx_buf[2 * NH + h], mx_buf[3 * NH + h]));
        float cor = 1.f;
        if (mx > m_used[v] + 8.f || m_used[v] == -INFINITY) {
          cor = m_used[v] == -INFINITY ? 0.f : exp2f(m_used[v] - mx);
          m_used[v] = mx;
          grew = true;
        }
        l_run[v] *= cor;
        my_vec[h] = m_used[v];
        my_cor[h] = cor;
      }
      __syncwarp();
      // the four warps see the same maxima, so they agree on whether to rescale
      if (i > 0 && __any_sync(0xffffffffu, grew)) {
        if (!mbar_wait_warp(o_done, (i - 1) & 1, abort_flag, g.status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
        tc_fence_after();
#pragma unroll 1
        for (int m = 0; m < n_blocks; ++m)
#pragma unroll 1
          for (int v = 0; v < NG; ++v) {
            uint32_t ov[32];
            tmem_ld32(tO + m * NH + v * 32 + lane_sel, ov);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) ov[e] = __float_as_uint(__uint_as_float(ov[e]) * my_cor[v * 32 + e]);
            tmem_st32(tO + m * NH + v * 32 + lane_sel, ov);
          }
        tmem_st_wait();
      }
      uint8_t* sP = sC + ((g.stages == 2 ? (i & 1) : 0) * g.na + g.na_lat) * kAtom + (r >> 6) * (NH * 128) + (r & 7) * 2;
      const int chunk = (r & 63) >> 3;
#pragma unroll
      for (int e = 0; e < NH; e += 4) {
        const float4 m4 = *reinterpret_cast<const float4*>(my_vec + e);
        sv[e] = exp2f(sv[e] - m4.x);            // -inf scores give zero; the maxima are finite
        sv[e + 1] = exp2f(sv[e + 1] - m4.y);
        sv[e + 2] = exp2f(sv[e + 2] - m4.z);
        sv[e + 3] = exp2f(sv[e + 3] - m4.w);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int h = e + x;
          *reinterpret_cast<bf16*>(sP + h * 128 + ((chunk ^ (h & 7)) << 4)) = __float2bfloat16_rn(sv[h]);
        }
      }
      fence_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
#pragma unroll
      for (int v = 0; v < NG; ++v) l_run[v] += halving_reduce<false>(sv + v * 32, lane);
    }
    if (ok && n_t > 0 && !mbar_wait_warp(o_done, (n_t - 1) & 1, abort_flag, g.status, kStatusWaitTimeoutEpilogue)) ok = false;
    tc_fence_after();
    // row sums of the four warps
    float* sums = s_cor;
#pragma unroll
    for (int v = 0; v < NG; ++v) my_cor[v * 32 + lane] = l_run[v];
    __syncwarp();
    if (ok) {
      if (lane == 0) mbar_arrive(warps_in);
      ok = mbar_wait_warp(warps_in, n_t & 1, abort_flag, g.status, kStatusWaitTimeoutEpilogue);
    }
#pragma unroll
    for (int v = 0; v < NG; ++v) {
      const int h = v * 32 + lane;
      const float l = (sums[h] + sums[NH + h]) + (sums[2 * NH + h] + sums[3 * NH + h]);
      float inv = 0.f;
      if (n_t > 0 && hb + h < a.heads) inv = 1.f / (a.sink ? l + exp2f(a.sink[hb + h] * kLog2e - m_used[v]) : l);
      my_vec[h] = n_splits == 1 ? inv : 1.f;
      if (n_splits > 1 && q == 0 && hb + h < a.heads) {
        float* ml = a.ws + ((static_cast<long long>(b) * a.heads + hb + h) * n_splits + split) * (a.rank + 2) + a.rank;
        ml[0] = m_used[v];
        ml[1] = l;
      }
    }
    __syncwarp();
    if (ok) {
#pragma unroll 1
      for (int m = 0; m < n_blocks; ++m)
#pragma unroll 1
        for (int v = 0; v < NG; ++v) {
          uint32_t ov[32];
          __syncwarp();
          if (n_t > 0) {
            tmem_ld32(tO + m * NH + v * 32 + lane_sel, ov);
            tmem_ld_wait();
          } else {
#pragma unroll
            for (int e = 0; e < 32; ++e) ov[e] = 0u;
          }
          const int d = m * 128 + r;
          if (d < a.rank) {
#pragma unroll
            for (int e = 0; e < 32; ++e) {
              const int h = hb + v * 32 + e;
              if (h >= a.heads) break;
              const float o = __uint_as_float(ov[e]) * my_vec[v * 32 + e];
              const long long oh = static_cast<long long>(b) * a.heads + h;
              if (n_splits == 1) static_cast<bf16*>(a.ctx)[oh * a.rank + d] = __float2bfloat16_rn(o);
              else a.ws[(oh * n_splits + split) * (a.rank + 2) + d] = o;
            }
          }
        }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(g.tmem_cols) : "memory");
  }
}

int heads_per_cta(const LatentDecodeArgs& a) {
  const int na = (a.rank + 63) / 64 + (a.rot + 63) / 64;
  return a.heads > 32 && na <= 9 ? 64 : 32;
}
size_t smem_bytes(int nh, int na, int stages) {
  return static_cast<size_t>(na) * nh * 128 + static_cast<size_t>(stages) * na * kAtom + (2 * 4 + 8) * nh * 4 + (6 + 4 * kMaxAtoms) * 8 + 16 + 1024;
}

template <int NH>
const char* launch(const LatentDecodeArgs& a, int n_splits, int* status, cudaStream_t s) {
  LatentTcGeom g{};
  g.na_lat = (a.rank + 63) / 64;
  g.na = g.na_lat + (a.rot + 63) / 64;
  g.stages = smem_bytes(NH, g.na, 2) <= 227 * 1024 ? 2 : 1;
  const int cols = ((g.na_lat + 1) / 2 + 2) * NH;
  g.tmem_cols = cols <= 128 ? 128 : (cols <= 256 ? 256 : 512);
  for (int k = 0; k < (a.rank + 15) / 16; ++k) g.kmask |= 1ull << k;
  for (int k = 0; k < (a.rot + 15) / 16; ++k) g.kmask |= 1ull << (4 * g.na_lat + k);
  g.status = status;
  const bf16* cache = static_cast<const bf16*>(a.cache);
  const long long row = static_cast<long long>(a.slots) * a.width;
  CUtensorMap tmC, tmCr, tmQ, tmQr;
  if (!make_map_3d(&tmC, cache, a.B, a.slots, a.rank, a.width, row, 1, kTok) ||
      !make_map_3d(&tmCr, cache + a.rank, a.B, a.slots, a.rot, a.width, row, 1, kTok) ||
      !make_map_3d(&tmQ, a.qa, a.B, a.heads, a.rank, a.rank, static_cast<long long>(a.heads) * a.rank, 1, NH) ||
      !make_map_3d(&tmQr, a.qr, a.B, a.heads, a.rot, a.qr_hs, a.ld_qr, 1, NH))
    return "latent_decode_tc: tensor map failed";
  auto kern = latent_decode_tc_kernel<NH>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) == cudaSuccess))
    return "latent_decode_tc: cannot reserve shared memory";
  if (launch_pdl(kern, dim3(n_splits, (a.heads + NH - 1) / NH, a.B), dim3(192), smem_bytes(NH, g.na, g.stages), s, tmC, tmCr, tmQ, tmQr, a,
                 n_splits, g) != cudaSuccess)
    return "latent_decode_tc launch failed";
  count_launch();
  return nullptr;
}

}  // namespace

bool latent_decode_tc_supported(const LatentDecodeArgs& a) {
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int na = (a.rank + 63) / 64 + (a.rot + 63) / 64;
  return a.dtype == kBF16 && a.rank % 8 == 0 && a.rank <= 512 && a.rot % 8 == 0 && na <= kMaxAtoms && a.width % 8 == 0 && a.ld_qr % 8 == 0 &&
         a.qr_hs % 8 == 0 && al16(a.qa) && al16(a.qr) && al16(a.cache) && smem_bytes(heads_per_cta(a), na, 1) <= 227 * 1024;
}

// key ranges per row: enough CTAs for the device, at least two tiles each
int latent_decode_splits(const LatentDecodeArgs& a, int num_sms) {
  const int nh = heads_per_cta(a), ctas = a.B * ((a.heads + nh - 1) / nh), tiles = (a.slots + kTok - 1) / kTok;
  return std::max(1, std::min({num_sms / std::max(ctas, 1), tiles / 2, 64}));
}

const char* latent_decode_tc(const LatentDecodeArgs& a, int n_splits, int* status, cudaStream_t s) {
  return heads_per_cta(a) == 64 ? launch<64>(a, n_splits, status, s) : launch<32>(a, n_splits, status, s);
}

}  // namespace ferrl
