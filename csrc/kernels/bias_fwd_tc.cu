// Sliding-window attention over whole sequences with a bias per distance and keys that are also the values
// (models/bias_attention.py), on the 5th-generation tensor cores.
//
// A CTA owns 128 queries of one head and walks the key tiles of its window:
//
//   S [128 x KT]  = Q K^T       the tile as TMA wrote it, K-major
//   O [128 x HD] += P K         the same bytes through an MN-major descriptor: a tile is fetched once and used twice
//
//   warp 0      TMA producer: Q once, then key tiles into a ring of four (zero-filled past the sequence and past a head's
//               own columns)
//   warp 1      tcgen05.mma issue; the scores of the next tile run under this tile's softmax, a tile goes back to the
//               producer when its P K has retired
//   warps 2-5   softmax, one query per thread, in base 2: s * scale + bias[distance].  Distances are constant along the
//               diagonals of a tile, so a warp's 32 queries need 31 + KT biases: a warp keeps two such slices in shared
//               memory, fetched a tile ahead, and lane l reads entry l + KT - 1 - key without bank conflicts.  P stays in
//               tensor memory as packed bf16; the output is rescaled only when a maximum grew by more than 2^8.
//
// Every wait is bounded and reports through the status word.
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

constexpr int kRows = 128;                      // queries per CTA
constexpr int kQAtom = kRows * 128;             // [128 x 64 columns] bf16
constexpr int kStages = 4;
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kBMajorMN = 1u << 16;        // instruction descriptor: B operand is MN-major

template <int NQ, int KT>
struct Cfg {
  static constexpr int HD = NQ * 64;
  static constexpr int K_ATOM = KT * 128, K_BYTES = NQ * K_ATOM;
  static constexpr int SLICE = 32 + KT;          // biases of one warp and tile (31 + KT used)
  static constexpr int SMEM = NQ * kQAtom + kStages * K_BYTES + 4 * 2 * SLICE * 4 + 256 + 1024;
  static_assert(3 * KT + HD <= 512, "tensor memory columns");
  static_assert(SMEM <= 227 * 1024, "shared memory");
};

template <int NQ, int KT>
__global__ void __launch_bounds__(192, 1)
bias_fwd_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, BiasFwdArgs a, int* status) {
  using C = Cfg<NQ, KT>;
  constexpr int HD = C::HD;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + NQ * kQAtom;
  float* s_bias = reinterpret_cast<float*>(sK + kStages * C::K_BYTES);      // [4 warps][2][SLICE]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_bias + 4 * 2 * C::SLICE);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;                   // [kStages]
  uint64_t* k_empty = k_full + kStages;          // [kStages]
  uint64_t* s_full = k_empty + kStages;          // [2]
  uint64_t* s_empty = s_full + 2;
  uint64_t* p_full = s_empty + 2;
  uint64_t* p_free = p_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(p_free + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_qt = (a.S + kRows - 1) / kRows;
  const int q0 = (n_qt - 1 - static_cast<int>(blockIdx.x)) * kRows;          // longest rows first
  const int hq = blockIdx.y, b = blockIdx.z, hk = hq / (a.Hq / a.Hkv);
  const int last_row = min(q0 + kRows, a.S) - 1;
  const int j_lo = max(0, q0 - a.window + 1) / KT;
  const int n_kv = last_row / KT - j_lo + 1;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < kStages; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], 4);
      mbar_init(&p_full[i], 4);
      mbar_init(&p_free[i], 1);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(512) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tS = tmem_base, tO = tmem_base + 2 * KT, tP = tO + HD;      // scores x 2, output, P x 2 (KT / 2 columns each)

  if (warp == 0) {
    if (lane == 0) {
      // ------------------------------------------------------------------ TMA producer
      mbar_expect_tx(q_full, NQ * kQAtom);
#pragma unroll
      for (int x = 0; x < NQ; ++x) tma_load_4d(sQ + x * kQAtom, &tmQ, q_full, x * 64, hq, q0, b);
      for (int i = 0; i < n_kv; ++i) {
        const int st = i % kStages;
        if (!mbar_wait(&k_empty[st], ((i / kStages) & 1) ^ 1, abort_flag, status, kStatusWaitTimeoutProducer)) break;
        mbar_expect_tx(&k_full[st], C::K_BYTES);
#pragma unroll
        for (int x = 0; x < NQ; ++x) tma_load_4d(sK + st * C::K_BYTES + x * C::K_ATOM, &tmK, &k_full[st], x * 64, hk, (j_lo + i) * KT, b);
      }
      if (*abort_flag) {
        for (int i = 0; i < 64; ++i) __nanosleep(10000);   // let copies in flight land before shared memory goes away
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA warp: all lanes walk the loop, one issues
    constexpr uint32_t idesc_s = make_idesc_bf16(128, KT), idesc_o = make_idesc_bf16(128, HD) | kBMajorMN;
    const uint64_t dq = make_smem_desc(smem_u32(sQ));
    auto issue_s = [&](int i) -> bool {
      const int st = i % kStages;
      if (!mbar_wait_warp(&k_full[st], (i / kStages) & 1, abort_flag, status, kStatusWaitTimeoutMma)) return false;
      if (!mbar_wait_warp(&s_empty[i & 1], ((i >> 1) & 1) ^ 1, abort_flag, status, kStatusWaitTimeoutMma)) return false;
      tc_fence_after();
      const uint64_t dk = make_smem_desc(smem_u32(sK + st * C::K_BYTES));
      const uint32_t ts = tS + (i & 1) * KT;
      if (elect_one()) {
#pragma unroll
        for (int k = 0; k < NQ * 4; ++k)
          umma(ts, desc_adv(dq, (k >> 2) * kQAtom + (k & 3) * 32), desc_adv(dk, (k >> 2) * C::K_ATOM + (k & 3) * 32), idesc_s, k > 0 ? 1u : 0u);
        umma_commit(&s_full[i & 1]);
      }
      __syncwarp();
      return true;
    };
    bool ok = mbar_wait_warp(q_full, 0, abort_flag, status, kStatusWaitTimeoutMma);
    if (ok) ok = issue_s(0);
    for (int i = 0; i < n_kv && ok; ++i) {
      if (i + 1 < n_kv) ok = issue_s(i + 1);
      if (!ok || !mbar_wait_warp(&p_full[i & 1], (i >> 1) & 1, abort_flag, status, kStatusWaitTimeoutMma)) break;
      tc_fence_after();
      const uint64_t dv = make_smem_desc_mn(smem_u32(sK + (i % kStages) * C::K_BYTES), C::K_ATOM);
      if (elect_one()) {
#pragma unroll
        for (int k = 0; k < KT / 16; ++k)
          umma_ts(tO, tP + (i & 1) * (KT / 2) + k * 8, desc_adv(dv, k * 2048), idesc_o, (i > 0 || k > 0) ? 1u : 0u);
        umma_commit(&p_free[i & 1]);
        umma_commit(&k_empty[i % kStages]);
      }
      __syncwarp();
    }
  } else {
    // ------------------------------------------------------------------ softmax and output (one query per thread)
    const int q = warp & 3, r = q * 32 + lane, row = q0 + r;
    const uint32_t lane_sel = static_cast<uint32_t>(q * 32) << 16;
    const float c = a.scale * kLog2e;
    const float* bias = a.bias + static_cast<long long>(hq) * a.bias_ld;
    float* slices = s_bias + q * 2 * C::SLICE;
    const int d_last = a.window - 1;
    constexpr int NB = C::SLICE / 32;
    float nb[NB];
    auto fetch = [&](int i) {                    // entry x of the slice: distance q0 + 32 q - k0 - (KT - 1) + x, clamped where it is masked anyway
      const int d0 = q0 + q * 32 - (j_lo + i) * KT - (KT - 1);
#pragma unroll
      for (int x = 0; x < NB; ++x) nb[x] = bias[min(max(d0 + x * 32 + lane, 0), d_last)] * kLog2e;
    };
    auto put = [&](int i) {
#pragma unroll
      for (int x = 0; x < NB; ++x) slices[(i & 1) * C::SLICE + x * 32 + lane] = nb[x];
      __syncwarp();
    };
    fetch(0);
    put(0);
    float m_used = -INFINITY, l_run = 0.f;
    const bool rows_ok = __all_sync(0xffffffffu, row < a.S);
    bool ok = true;
    for (int i = 0; i < n_kv; ++i) {
      const int st = i & 1;
      if (i + 1 < n_kv) fetch(i + 1);
      if (!mbar_wait_warp(&s_full[st], (i >> 1) & 1, abort_flag, status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
      tc_fence_after();
      uint32_t sv[KT];
#pragma unroll
      for (int cc = 0; cc < KT; cc += 32) tmem_ld32(tS + st * KT + lane_sel + cc, sv + cc);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_empty[st]);
      const float* sl = slices + st * C::SLICE + lane + KT - 1;
#pragma unroll
      for (int e = 0; e < KT; ++e) sv[e] = __float_as_uint(__uint_as_float(sv[e]) * c + sl[-e]);
      const int k0 = (j_lo + i) * KT;
      // warp-uniform: no row of the CTA is cut by the diagonal, the window's lower edge or the sequence end
      const bool full = rows_ok && k0 + KT - 1 <= q0 && q0 + kRows - a.window <= k0;
      if (!full) {
        const int limit = min(a.S, row + 1) - k0, lo = row - a.window + 1 - k0;      // keys [lo, limit) of the tile are visible
#pragma unroll
        for (int e = 0; e < KT; ++e)
          if (e >= limit || e < lo) sv[e] = __float_as_uint(-INFINITY);
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int e = 0; e < KT; ++e) mx4[e & 3] = fmaxf(mx4[e & 3], __uint_as_float(sv[e]));
      const float m_new = fmaxf(m_used, fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])));
      const bool need = i > 0 && m_new > m_used && (m_used == -INFINITY || m_new - m_used > 8.f);
      if (i == 0) m_used = m_new;
      if (__any_sync(0xffffffffu, need)) {
        if (!mbar_wait_warp(&p_free[(i - 1) & 1], ((i - 1) >> 1) & 1, abort_flag, status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
        tc_fence_after();
        const float corr = need ? (m_used == -INFINITY ? 0.f : exp2f(m_used - m_new)) : 1.f;
        if (need) {
          m_used = m_new;
          l_run *= corr;
        }
#pragma unroll 1
        for (int cc = 0; cc < HD; cc += 32) {
          uint32_t ov[32];
          tmem_ld32(tO + lane_sel + cc, ov);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; ++e) ov[e] = __float_as_uint(__uint_as_float(ov[e]) * corr);
          tmem_st32(tO + lane_sel + cc, ov);
        }
        tmem_st_wait();
        tc_fence_before();
      }
      // P[st] is free again once P K of tile i - 2 has retired
      if (i >= 2 && !mbar_wait_warp(&p_free[st], ((i >> 1) - 1) & 1, abort_flag, status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
      const float mc = m_used == -INFINITY ? 0.f : m_used;      // nothing visible yet: every score is -inf and gives zero
      float ps4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int e = 0; e < KT; e += 2) {
        const float p0 = exp2f(__uint_as_float(sv[e]) - mc), p1 = exp2f(__uint_as_float(sv[e + 1]) - mc);
        ps4[(e >> 1) & 3] += p0 + p1;
        __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
        sv[e >> 1] = *reinterpret_cast<uint32_t*>(&h);
      }
      l_run += (ps4[0] + ps4[1]) + (ps4[2] + ps4[3]);
#pragma unroll
      for (int cc = 0; cc < KT / 2; cc += 32) tmem_st32(tP + st * (KT / 2) + lane_sel + cc, sv + cc);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[st]);
      if (i + 1 < n_kv) put(i + 1);
    }
    // the last P K completes the output
    if (ok && !mbar_wait_warp(&p_free[(n_kv - 1) & 1], ((n_kv - 1) >> 1) & 1, abort_flag, status, kStatusWaitTimeoutEpilogue)) ok = false;
    tc_fence_after();
    if (ok) {      // warp-uniform: the TMEM loads are warp-collective, only the stores are per row
      const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
      bf16* orow = static_cast<bf16*>(a.out) + (static_cast<long long>(b) * a.S + row) * a.Hq * a.D + static_cast<long long>(hq) * a.D;
#pragma unroll 1
      for (int cc = 0; cc < HD; cc += 32) {
        uint32_t ov[32];
        __syncwarp();   // lanes that skipped the stores rejoin before the collective load
        tmem_ld32(tO + lane_sel + cc, ov);
        tmem_ld_wait();
        if (row < a.S) {
#pragma unroll
          for (int ch = 0; ch < 4; ++ch) {
            if (cc + ch * 8 >= a.D) break;
            uint4 w;
            __nv_bfloat162* wh = reinterpret_cast<__nv_bfloat162*>(&w);
#pragma unroll
            for (int e = 0; e < 4; ++e)
              wh[e] = __floats2bfloat162_rn(__uint_as_float(ov[ch * 8 + 2 * e]) * inv, __uint_as_float(ov[ch * 8 + 2 * e + 1]) * inv);
            reinterpret_cast<uint4*>(orow + cc)[ch] = w;
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(512) : "memory");
  }
}

template <int NQ, int KT>
const char* launch(const BiasFwdArgs& a, int* status, cudaStream_t s) {
  CUtensorMap tmQ, tmK;
  if (!make_map_4d(&tmQ, a.q, a.B, a.S, a.Hq, a.D, a.D, a.q_ts, a.q_bs, kRows) || !make_map_4d(&tmK, a.k, a.B, a.S, a.Hkv, a.D, a.D, a.k_ts, a.k_bs, KT))
    return "bias_fwd_tc: tensor map failed";
  auto k = bias_fwd_tc_kernel<NQ, KT>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<NQ, KT>::SMEM) == cudaSuccess))
    return "bias_fwd_tc: cannot reserve shared memory";
  k<<<dim3((a.S + kRows - 1) / kRows, a.Hq, a.B), 192, Cfg<NQ, KT>::SMEM, s>>>(tmQ, tmK, a, status);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "bias_fwd_tc launch failed";
}

}  // namespace

bool bias_fwd_tc_supported(const BiasFwdArgs& a) {
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return a.dtype == kBF16 && a.D % 8 == 0 && a.D <= 256 && a.q_ts % 8 == 0 && a.q_bs % 8 == 0 && a.k_ts % 8 == 0 && a.k_bs % 8 == 0 && al16(a.q) &&
         al16(a.k) && al16(a.out);
}

const char* bias_fwd_tc(const BiasFwdArgs& a, int* status, cudaStream_t s) {
  if (!bias_fwd_tc_supported(a)) return "bias_fwd_tc: unsupported arguments";
  if (a.B == 0 || a.S == 0) return nullptr;
  switch ((a.D + 63) / 64) {
    case 1: return launch<1, 128>(a, status, s);
    case 2: return launch<2, 128>(a, status, s);
    case 3: return launch<3, 64>(a, status, s);
    default: return launch<4, 64>(a, status, s);
  }
}

}  // namespace ferrl
