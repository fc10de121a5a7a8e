// One query per row against a ring of cached keys that are also the values, scores with a bias per distance
// (models/bias_attention.py), on the 5th-generation tensor cores.
//
// A CTA owns one row, one key head, up to NH of its query heads and a range of the ring, in tiles of 128 slots.  As in
// latent_decode_tc.cu the products run transposed, so that the 128 rows of an MMA are slots or key entries, never heads:
//
//   S^T [128 slots x NH]    = K Q^T         the tile as TMA wrote it, K-major
//   O^T [128 entries x NH] += K^T P         the same bytes through an MN-major descriptor
//
// so every cached byte crosses the memory system once.
//
//   warp 0      TMA producer.  The CTA whose range holds the token's own slot stores its key there first (generic stores,
//               proxy fence, then the copies).
//   warp 1      tcgen05.mma issue: the next tile's scores run under this tile's softmax
//   warps 2-5   softmax, one slot per thread, HP heads each (the MMA's NH rounded up from them; the padding's weights are
//               zeros written once).  Biases come straight from the table, distances fall from lane to lane.  Maxima and
//               sums over the slots by a halving exchange inside the warp and a small shared array between the warps.
//
// Several ranges of a row are joined by attn_combine.  Every wait is bounded and reports through the status word.
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

constexpr int kTok = 128;                       // slots per tile
constexpr int kAtom = kTok * 128;               // [128 slots x 64 columns] bf16: 16 KB
constexpr int kMaxStages = 6;
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kAMajorMN = 1u << 15;        // instruction descriptor: A operand is MN-major

template <int NH> __device__ __forceinline__ void tmem_ld_heads(uint32_t taddr, uint32_t* r) {
  if constexpr (NH == 32) {
    tmem_ld32(taddr, r);
  } else {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
          "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(taddr)
        : "memory");
  }
}
template <int NH> __device__ __forceinline__ void tmem_st_heads(uint32_t taddr, const uint32_t* r) {
  if constexpr (NH == 32) {
    tmem_st32(taddr, r);
  } else {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
          "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
        : "memory");
  }
}

// HP values per lane, reduced over the 32 lanes: every lane returns the result of value (lane mod HP)
template <int HP, bool MAX>
__device__ __forceinline__ float lanes_reduce(const float* in, int lane) {
  float v[HP];
#pragma unroll
  for (int j = 0; j < HP; ++j) v[j] = in[j];
#pragma unroll
  for (int w = HP / 2; w >= 1; w >>= 1) {
    const bool up = (lane & w) != 0;
#pragma unroll
    for (int j = 0; j < w; ++j) {
      const float send = up ? v[j] : v[j + w], keep = up ? v[j + w] : v[j];
      const float got = __shfl_xor_sync(0xffffffffu, send, w);
      v[j] = MAX ? fmaxf(keep, got) : keep + got;
    }
  }
#pragma unroll
  for (int w = HP; w < 32; w <<= 1) {
    const float got = __shfl_xor_sync(0xffffffffu, v[0], w);
    v[0] = MAX ? fmaxf(v[0], got) : v[0] + got;
  }
  return v[0];
}

struct Geom {
  int na, stages, tmem_cols, k_steps;           // 64-column atoms of a key, tiles in shared memory
  int* status;
};

template <int NH, int HP>
__global__ void __launch_bounds__(192, NH == 32 ? 1 : (HP <= 4 ? 3 : 2))
bias_decode_tc_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmQ, BiasDecodeArgs a, int n_splits, Geom geo) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int tile_bytes = geo.na * kAtom;
  uint8_t* sK = smem;
  uint8_t* sQ = sK + geo.stages * tile_bytes;
  uint8_t* sP = sQ + geo.na * (NH * 128);       // [2 atoms][NH x 64 slots]
  float* s_max = reinterpret_cast<float*>(sP + 2 * NH * 128);       // [2 tiles][4 warps][HP]
  float* s_vec = s_max + 2 * 4 * HP;            // [4 warps][NH] maxima in use, at the end 1 / denominator
  float* s_cor = s_vec + 4 * NH;                // [4 warps][NH] rescale factors, at the end the row sums
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_cor + 4 * NH);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;                  // [2]
  uint64_t* p_full = bars + 3;
  uint64_t* o_done = bars + 4;
  uint64_t* warps_in = bars + 5;                // the four softmax warps meet here once a tile and once at the end
  uint64_t* full = bars + 6;                    // [stages]
  uint64_t* empty = full + kMaxStages;          // [stages]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(empty + kMaxStages);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rep = a.Hq / a.Hkv, head_tiles = (rep + NH - 1) / NH;
  const int split = blockIdx.x, g = blockIdx.y / head_tiles, h0 = (blockIdx.y % head_tiles) * NH, b = blockIdx.z;
  const int nh = min(NH, rep - h0), hq0 = g * rep + h0, D = a.D;
  const int n_blocks = (geo.na + 1) / 2;        // 128-entry blocks of a key
  pdl_trigger();
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    mbar_init(p_full, 4);
    mbar_init(o_done, 1);
    mbar_init(warps_in, 4);
    for (int i = 0; i < geo.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(geo.tmem_cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if constexpr (HP < NH) {
    for (int i = threadIdx.x; i < 2 * NH * 8; i += 192) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0, 0, 0, 0);
    fence_async_smem();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_wait();                                   // positions, queries and the token's key come from the predecessors
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tO = tmem_base, tS = tmem_base + n_blocks * NH;           // S^T buffers at tS and tS + NH
  const bool on = !a.active || a.active[b];
  const int pos = a.kv_len[b];
  const int n = on ? min(pos + 1, a.slots) : 0, cur = pos % a.slots;
  const int tiles = (n + kTok - 1) / kTok;
  const int t_lo = static_cast<int>(static_cast<long long>(tiles) * split / n_splits);
  const int n_t = static_cast<int>(static_cast<long long>(tiles) * (split + 1) / n_splits) - t_lo;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (cur >= t_lo * kTok && cur < (t_lo + n_t) * kTok) {
      const long long row = static_cast<long long>(a.Hkv) * D;
      bf16* dst = static_cast<bf16*>(a.cache) + (static_cast<long long>(b) * a.slots + cur) * row + static_cast<long long>(g) * D;
      const bf16* src = static_cast<const bf16*>(a.k) + b * a.ld_k + static_cast<long long>(g) * D;
      if (lane < D / 8) reinterpret_cast<uint4*>(dst)[lane] = reinterpret_cast<const uint4*>(src)[lane];
      asm volatile("fence.proxy.async;" ::: "memory");
      __syncwarp();
    }
    if (lane == 0 && n_t > 0) {
      mbar_expect_tx(q_full, geo.na * NH * 128);
      for (int x = 0; x < geo.na; ++x) tma_load_3d(sQ + x * (NH * 128), &tmQ, q_full, x * 64, hq0, b);
      for (int i = 0; i < n_t; ++i) {
        const int st = i % geo.stages, use = i / geo.stages;
        if (use > 0 && !mbar_wait(&empty[st], (use - 1) & 1, abort_flag, geo.status, kStatusWaitTimeoutProducer)) break;
        mbar_expect_tx(&full[st], tile_bytes);
        for (int x = 0; x < geo.na; ++x) tma_load_4d(sK + st * tile_bytes + x * kAtom, &tmK, &full[st], x * 64, g, (t_lo + i) * kTok, b);
      }
      if (*abort_flag) {
        for (int i = 0; i < 64; ++i) __nanosleep(10000);   // let copies in flight land before shared memory goes away
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA warp: all lanes walk the loop, one issues
    constexpr uint32_t idesc_s = make_idesc_bf16(128, NH), idesc_o = make_idesc_bf16(128, NH) | kAMajorMN;
    const uint64_t dq = make_smem_desc(smem_u32(sQ)), dp = make_smem_desc(smem_u32(sP));
    auto issue_s = [&](int i) -> bool {
      const int st = i % geo.stages;
      if (!mbar_wait_warp(&full[st], (i / geo.stages) & 1, abort_flag, geo.status, kStatusWaitTimeoutMma)) return false;
      tc_fence_after();
      const uint64_t dk = make_smem_desc(smem_u32(sK + st * tile_bytes));
      if (elect_one()) {
        for (int k = 0; k < geo.k_steps; ++k)
          umma(tS + (i & 1) * NH, desc_adv(dk, (k >> 2) * kAtom + (k & 3) * 32), desc_adv(dq, (k >> 2) * (NH * 128) + (k & 3) * 32), idesc_s, k > 0 ? 1u : 0u);
        umma_commit(&s_full[i & 1]);
      }
      __syncwarp();
      return true;
    };
    bool ok = n_t > 0 && mbar_wait_warp(q_full, 0, abort_flag, geo.status, kStatusWaitTimeoutMma);
    if (ok) ok = issue_s(0);
    for (int i = 0; i < n_t && ok; ++i) {
      // S^T buffer (i + 1) & 1 is free: its last reader announced P of tile i - 1, which has been waited for
      if (i + 1 < n_t) ok = issue_s(i + 1);
      if (!ok || !mbar_wait_warp(p_full, i & 1, abort_flag, geo.status, kStatusWaitTimeoutMma)) break;
      tc_fence_after();
      const int st = i % geo.stages;
      for (int m = 0; m < n_blocks; ++m) {
        const uint64_t dk = make_smem_desc_mn(smem_u32(sK + st * tile_bytes + 2 * m * kAtom), kAtom);
        if (elect_one()) {
#pragma unroll
          for (int k = 0; k < kTok / 16; ++k)
            umma(tO + m * NH, desc_adv(dk, k * 2048), desc_adv(dp, (k >> 2) * (NH * 128) + (k & 3) * 32), idesc_o, (i > 0 || k > 0) ? 1u : 0u);
          if (m == n_blocks - 1) {
            umma_commit(&empty[st]);
            umma_commit(o_done);
          }
        }
        __syncwarp();
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax and output
    const int q = warp & 3, r = q * 32 + lane;  // slot inside the tile == tensor-memory lane
    const uint32_t lane_sel = static_cast<uint32_t>(q * 32) << 16;
    const float c2 = a.scale * kLog2e;
    const float* bias = a.bias + static_cast<long long>(hq0) * a.bias_ld;
    const int hl = lane % HP;                   // this lane's head in the reductions
    float m_used = -INFINITY, l_run = 0.f;      // of head hl, the same in all four warps (maxima) or this warp's share (sums)
    float* my_vec = s_vec + q * NH;
    float* my_cor = s_cor + q * NH;
    bool ok = true;
    float bv[HP];                               // biases of this thread's slot, fetched a tile ahead
    auto fetch = [&](int i) {
      const int slot = (t_lo + i) * kTok + r;
      const int d = slot < n ? (cur >= slot ? cur - slot : cur - slot + a.slots) : 0;
#pragma unroll
      for (int e = 0; e < HP; ++e) bv[e] = e < nh ? __ldg(bias + e * a.bias_ld + d) : 0.f;
    };
    if (n_t > 0) fetch(0);
    for (int i = 0; i < n_t; ++i) {
      const bool live = (t_lo + i) * kTok + r < n;
      if (!mbar_wait_warp(&s_full[i & 1], (i >> 1) & 1, abort_flag, geo.status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
      tc_fence_after();
      float sv[NH];
      tmem_ld_heads<NH>(tS + (i & 1) * NH + lane_sel, reinterpret_cast<uint32_t*>(sv));
      tmem_ld_wait();
#pragma unroll
      for (int e = 0; e < HP; ++e) sv[e] = live ? sv[e] * c2 + bv[e] * kLog2e : -INFINITY;
      if (i + 1 < n_t) fetch(i + 1);
      float* mx_buf = s_max + (i & 1) * 4 * HP;
      const float wm = lanes_reduce<HP, true>(sv, lane);
      if (lane < HP) mx_buf[q * HP + lane] = wm;
      __syncwarp();
      if (lane == 0) mbar_arrive(warps_in);
      if (!mbar_wait_warp(warps_in, i & 1, abort_flag, geo.status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
      const float mx = fmaxf(fmaxf(mx_buf[hl], mx_buf[HP + hl]), fmaxf(mx_buf[2 * HP + hl], mx_buf[3 * HP + hl]));
      float cor = 1.f;
      bool grew = false;
      if (mx > m_used + 8.f || m_used == -INFINITY) {
        cor = m_used == -INFINITY ? 0.f : exp2f(m_used - mx);
        m_used = mx;
        grew = true;
      }
      l_run *= cor;
      if (lane < HP) {
        my_vec[lane] = m_used;
        my_cor[lane] = cor;
      }
      __syncwarp();
      // the tile before has been added up: its weights may be overwritten and the sums rescaled
      if (i > 0 && !mbar_wait_warp(o_done, (i - 1) & 1, abort_flag, geo.status, kStatusWaitTimeoutEpilogue)) { ok = false; break; }
      // the four warps see the same maxima, so they agree on whether to rescale
      if (i > 0 && __any_sync(0xffffffffu, grew)) {
        tc_fence_after();
#pragma unroll 1
        for (int m = 0; m < n_blocks; ++m) {
          uint32_t ov[NH];
          tmem_ld_heads<NH>(tO + m * NH + lane_sel, ov);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < HP; ++e) ov[e] = __float_as_uint(__uint_as_float(ov[e]) * my_cor[e]);
          tmem_st_heads<NH>(tO + m * NH + lane_sel, ov);
        }
        tmem_st_wait();
      }
      uint8_t* p = sP + (r >> 6) * (NH * 128) + (r & 7) * 2;
      const int chunk = (r & 63) >> 3;
#pragma unroll
      for (int e = 0; e < HP; ++e) {
        sv[e] = exp2f(sv[e] - my_vec[e]);       // -inf scores give zero; the maxima are finite
        *reinterpret_cast<bf16*>(p + e * 128 + ((chunk ^ (e & 7)) << 4)) = __float2bfloat16_rn(sv[e]);
      }
      fence_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
      l_run += lanes_reduce<HP, false>(sv, lane);
    }
    if (ok && n_t > 0 && !mbar_wait_warp(o_done, (n_t - 1) & 1, abort_flag, geo.status, kStatusWaitTimeoutEpilogue)) ok = false;
    tc_fence_after();
    // row sums of the four warps
    if (lane < HP) my_cor[lane] = l_run;
    __syncwarp();
    if (ok) {
      if (lane == 0) mbar_arrive(warps_in);
      ok = mbar_wait_warp(warps_in, n_t & 1, abort_flag, geo.status, kStatusWaitTimeoutEpilogue);
    }
    const float l = (s_cor[hl] + s_cor[NH + hl]) + (s_cor[2 * NH + hl] + s_cor[3 * NH + hl]);
    if (lane < HP) my_vec[lane] = n_splits > 1 ? 1.f : (n_t > 0 ? 1.f / l : 0.f);
    if (n_splits > 1 && q == 0 && lane < nh) {
      float* ml = a.ws + ((static_cast<long long>(b) * a.Hq + hq0 + lane) * n_splits + split) * (D + 2) + D;
      ml[0] = m_used;
      ml[1] = l;
    }
    __syncwarp();
    if (ok) {
#pragma unroll 1
      for (int m = 0; m < n_blocks; ++m) {
        uint32_t ov[NH];
        __syncwarp();
        if (n_t > 0) {
          tmem_ld_heads<NH>(tO + m * NH + lane_sel, ov);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int e = 0; e < NH; ++e) ov[e] = 0u;
        }
        const int d = m * 128 + r;
        if (d < D) {
#pragma unroll
          for (int e = 0; e < HP; ++e) {
            if (e >= nh) break;
            const float o = __uint_as_float(ov[e]) * my_vec[e];
            const long long oh = static_cast<long long>(b) * a.Hq + hq0 + e;
            if (n_splits == 1) static_cast<bf16*>(a.out)[oh * D + d] = __float2bfloat16_rn(o);
            else a.ws[(oh * n_splits + split) * (D + 2) + d] = o;
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(geo.tmem_cols) : "memory");
  }
}

// With an odd number of atoms the last 128-entry block of K^T P reads one atom past its tile (its rows go nowhere), which
// for the last tile must still be this CTA's memory.
size_t smem_bytes(int nh, int na, int stages) {
  const size_t tiles = static_cast<size_t>(stages) * na * kAtom;
  const size_t rest = static_cast<size_t>(na) * nh * 128 + 2 * nh * 128 + (2 * 4 * 32 + 8 * nh) * 4 + (6 + 2 * kMaxStages) * 8 + 16;
  return tiles + (na % 2 ? std::max<size_t>(rest, kAtom) : rest) + 1024;
}
// tiles in shared memory: at least two, and as many as leave room for three CTAs on an SM, else two, else one
int stages_of(int nh, int na) {
  for (int ctas = 3; ctas >= 1; --ctas)
    for (int st = kMaxStages; st >= 2; --st)
      if (smem_bytes(nh, na, st) + 1024 <= static_cast<size_t>(228 * 1024) / ctas) return st;
  return 2;
}
int heads_per_cta(const BiasDecodeArgs& a) { return a.Hq / a.Hkv > 16 ? 32 : 16; }

template <int NH, int HP>
const char* launch(const BiasDecodeArgs& a, int n_splits, int* status, cudaStream_t s) {
  Geom geo{};
  geo.na = (a.D + 63) / 64;
  geo.k_steps = (a.D + 15) / 16;
  geo.stages = stages_of(NH, geo.na);
  const int cols = ((geo.na + 1) / 2 + 2) * NH;
  geo.tmem_cols = cols <= 64 ? 64 : 128;
  geo.status = status;
  const long long row = static_cast<long long>(a.Hkv) * a.D;
  CUtensorMap tmK, tmQ;
  if (!make_map_4d(&tmK, a.cache, a.B, a.slots, a.Hkv, a.D, a.D, row, a.slots * row, kTok) ||
      !make_map_3d(&tmQ, a.q, a.B, a.Hq, a.D, a.D, a.ld_q, 1, NH))
    return "bias_decode_tc: tensor map failed";
  auto k = bias_decode_tc_kernel<NH, HP>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) == cudaSuccess))
    return "bias_decode_tc: cannot reserve shared memory";
  const int rep = a.Hq / a.Hkv;
  if (launch_pdl(k, dim3(n_splits, a.Hkv * ((rep + NH - 1) / NH), a.B), dim3(192), smem_bytes(NH, geo.na, geo.stages), s, tmK, tmQ, a, n_splits, geo) !=
      cudaSuccess)
    return "bias_decode_tc launch failed";
  count_launch();
  return nullptr;
}

}  // namespace

bool bias_decode_tc_supported(const BiasDecodeArgs& a) {
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return a.dtype == kBF16 && a.D % 8 == 0 && a.D <= 256 && a.ld_k % 8 == 0 && a.ld_q % 8 == 0 && al16(a.q) && al16(a.k) && al16(a.cache);
}

// ranges of a row: enough CTAs for the device, at least two tiles each
int bias_decode_splits(const BiasDecodeArgs& a, int num_sms) {
  const int nh = heads_per_cta(a), rep = a.Hq / a.Hkv, ctas = std::max(1, a.B * a.Hkv * ((rep + nh - 1) / nh));
  return std::max(1, std::min({2 * num_sms / ctas, a.slots / (2 * kTok), 32}));
}

const char* bias_decode_tc(const BiasDecodeArgs& a, int n_splits, int* status, cudaStream_t s) {
  if (!bias_decode_tc_supported(a)) return "bias_decode_tc: unsupported arguments";
  if (a.B == 0) return nullptr;
  if (n_splits > 1 && !a.ws) return "bias_decode_tc: workspace missing";
  const int rep = a.Hq / a.Hkv;
  const char* err = rep > 16 ? launch<32, 32>(a, n_splits, status, s) : rep > 8 ? launch<16, 16>(a, n_splits, status, s)
                  : rep > 4  ? launch<16, 8>(a, n_splits, status, s) : launch<16, 4>(a, n_splits, status, s);
  if (err) return err;
  if (n_splits > 1) return attn_combine(a.ws, nullptr, a.out, static_cast<long long>(a.B) * a.Hq, a.Hq, a.D, n_splits, s);
  return cudaGetLastError() == cudaSuccess ? nullptr : "bias_decode_tc launch failed";
}

}  // namespace ferrl
