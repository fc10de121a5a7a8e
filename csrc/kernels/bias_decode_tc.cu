// One query per row against a ring of cached keys that are also the values, scores with a bias per distance
// (models/bias_attention.py), bf16 on the warp-level tensor path.
//
// A CTA owns one row, one key head and up to 16 of its query heads, and a range of the ring's slots.  Its four warps walk
// blocks of 16 slots on their own, each through a private ring of cp.async stages, and meet only at the end:
//
//   S [16 heads x 16 slots] = Q K^T       K: the block's rows as fetched, one ldmatrix per 16 x 16 piece
//   O [16 heads x D]       += P K         the same bytes through ldmatrix.trans
//
// so every cached byte crosses the memory system once and shared memory twice.  The biases of a block travel with it.
// The token's own key is read from the projection wherever its slot comes up, and one CTA stores it.  Several ranges of a
// row are joined by attn_combine.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <algorithm>

#include "../api.h"
#include "../common.cuh"
#include "mma_sync.cuh"

namespace ferrl {
namespace {

using namespace mmah;
using bf16 = __nv_bfloat16;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kWarps = 4, kKeys = 16, kStages = 4, kHeads = 16;

__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src, bool valid) {
  const int sz = valid ? 4 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(sz) : "memory");
}

template <int KD>
struct Cfg {
  static constexpr int DP = KD * 16, ROW = DP * 2 + 16;           // an odd number of 16-byte chunks: conflict-free ldmatrix
  static constexpr int STAGE = kKeys * ROW + kHeads * kKeys * 4;  // keys, then biases [head][slot]
  static constexpr int SMEM = kWarps * kStages * STAGE;
  static_assert(SMEM >= kWarps * kHeads * (DP + 2) * 4, "the merge reuses the stages");
};

template <int KD>
__global__ void __launch_bounds__(kWarps * 32) bias_decode_tc_kernel(BiasDecodeArgs a, int n_splits) {
  using C = Cfg<KD>;
  extern __shared__ __align__(16) uint8_t bd_smem[];
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rep = a.Hq / a.Hkv, head_tiles = (rep + kHeads - 1) / kHeads;
  const int split = blockIdx.x, g = blockIdx.y / head_tiles, h0 = (blockIdx.y % head_tiles) * kHeads, b = blockIdx.z;
  const int nh = min(kHeads, rep - h0), hq0 = g * rep + h0, D = a.D;
  pdl_wait();
  const bool on = !a.active || a.active[b];
  const int pos = a.kv_len[b];
  const int n = on ? min(pos + 1, a.slots) : 0, cur = pos % a.slots;
  const int blocks = (n + kKeys * kWarps - 1) / (kKeys * kWarps);
  const int lo = static_cast<int>(static_cast<long long>(blocks) * split / n_splits) * kKeys * kWarps;
  const int hi = min(n, static_cast<int>(static_cast<long long>(blocks) * (split + 1) / n_splits) * kKeys * kWarps);
  const long long row = static_cast<long long>(a.Hkv) * D;
  bf16* cache = static_cast<bf16*>(a.cache) + static_cast<long long>(b) * a.slots * row + static_cast<long long>(g) * D;
  const bf16* kn = static_cast<const bf16*>(a.k) + b * a.ld_k + static_cast<long long>(g) * D;
  const bf16* q = static_cast<const bf16*>(a.q) + b * a.ld_q + static_cast<long long>(hq0) * D;
  const float* bias = a.bias + static_cast<long long>(hq0) * a.bias_ld;
  if (on && split == 0 && h0 == 0)
    for (int i = threadIdx.x; i < D / 8; i += kWarps * 32)
      reinterpret_cast<uint4*>(cache + cur * row)[i] = reinterpret_cast<const uint4*>(kn)[i];

  const uint32_t ring = smem_addr(bd_smem) + warp * kStages * C::STAGE;
  const int n_it = lo < hi ? (hi - lo + kKeys * kWarps - 1) / (kKeys * kWarps) : 0;
  auto issue = [&](int it) {
    if (it < n_it) {
      const uint32_t st = ring + (it % kStages) * C::STAGE;
      const int j0 = lo + (it * kWarps + warp) * kKeys;
      constexpr int CPR = C::DP / 8;
#pragma unroll 4
      for (int c = lane; c < kKeys * CPR; c += 32) {
        const int r = c / CPR, part = c - r * CPR, j = j0 + r;
        const bool ok = j < hi && part * 8 < D;
        const bf16* src = ok ? (j == cur ? kn : cache + j * row) + part * 8 : kn;
        cp_async16(st + r * C::ROW + part * 16, src, ok);
      }
      for (int c = lane; c < nh * kKeys; c += 32) {
        const int h = c / kKeys, j = j0 + (c & (kKeys - 1));
        const bool ok = j < hi;
        const int d = cur >= j ? cur - j : cur - j + a.slots;
        cp_async4(st + kKeys * C::ROW + c * 4, ok ? bias + h * a.bias_ld + d : bias, ok);
      }
    }
    cp_commit();
  };
#pragma unroll
  for (int s = 0; s < kStages - 1; ++s) issue(s);

  const int gr = lane >> 2, t = lane & 3;
  uint32_t qa[KD][4];
#pragma unroll
  for (int ks = 0; ks < KD; ++ks)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = gr + (e & 1) * 8, c = ks * 16 + 2 * t + (e >> 1) * 8;
      qa[ks][e] = r < nh && c < D ? *reinterpret_cast<const uint32_t*>(q + static_cast<long long>(r) * D + c) : 0u;
    }
  float o[2 * KD][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2 * KD; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const float c2 = a.scale * kLog2e;
  const int kr = (lane & 7) + ((lane >> 4) << 3), kc = (lane >> 3) & 1;      // scores: rows are slots, chunks the contraction
  const int vr = lane & 15, vc = lane >> 4;                                  // output: rows the contraction, chunks columns
  for (int it = 0; it < n_it; ++it) {
    cp_wait<kStages - 2>();
    __syncwarp();
    issue(it + kStages - 1);
    const uint32_t st = ring + (it % kStages) * C::STAGE;
    const float* sb = reinterpret_cast<const float*>(bd_smem + (st - smem_addr(bd_smem)) + kKeys * C::ROW);
    const int j0 = lo + (it * kWarps + warp) * kKeys;
    float s[2][4];
#pragma unroll
    for (int e = 0; e < 4; ++e) s[0][e] = s[1][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < KD; ++ks) {
      uint32_t b0, b1, b2, b3;
      ldsm4(st + kr * C::ROW + (ks * 2 + kc) * 16, b0, b1, b2, b3);
      mma16816(s[0], qa[ks], b0, b1);
      mma16816(s[1], qa[ks], b2, b3);
    }
    float mn[2] = {m[0], m[1]};
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = x * 8 + 2 * t + (e & 1), h = gr + (e >> 1) * 8;
        const bool ok = j0 + key < hi && h < nh;
        s[x][e] = ok ? s[x][e] * c2 + sb[h * kKeys + key] * kLog2e : -INFINITY;
        mn[e >> 1] = fmaxf(mn[e >> 1], s[x][e]);
      }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mn[i] = fmaxf(mn[i], __shfl_xor_sync(0xffffffffu, mn[i], 1));
      mn[i] = fmaxf(mn[i], __shfl_xor_sync(0xffffffffu, mn[i], 2));
    }
    if (__any_sync(0xffffffffu, mn[0] > m[0] || mn[1] > m[1])) {
      float cor[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        cor[i] = m[i] == -INFINITY ? 0.f : exp2f(m[i] - mn[i]);
        l[i] *= cor[i];
        m[i] = mn[i];
      }
#pragma unroll
      for (int i = 0; i < 2 * KD; ++i) {
        o[i][0] *= cor[0];
        o[i][1] *= cor[0];
        o[i][2] *= cor[1];
        o[i][3] *= cor[1];
      }
    }
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float p = s[x][e] == -INFINITY ? 0.f : exp2f(s[x][e] - m[e >> 1]);
        s[x][e] = p;
        l[e >> 1] += p;
      }
    const uint32_t pa[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
#pragma unroll
    for (int nt = 0; nt < KD; ++nt) {
      uint32_t b0, b1, b2, b3;
      ldsm4t(st + vr * C::ROW + (nt * 2 + vc) * 16, b0, b1, b2, b3);
      mma16816(o[2 * nt], pa, b0, b1);
      mma16816(o[2 * nt + 1], pa, b2, b3);
    }
    __syncwarp();                       // everyone is done with the stage that is filled next
  }
  cp_wait<0>();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
  }
  __syncthreads();
  // merge of the warps: [warp][head][DP] outputs, then maxima and sums
  float* so = reinterpret_cast<float*>(bd_smem);
  float* sm = so + kWarps * kHeads * C::DP;
  float* sl = sm + kWarps * kHeads;
#pragma unroll
  for (int i = 0; i < 2 * KD; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) so[(warp * kHeads + gr + (e >> 1) * 8) * C::DP + i * 8 + 2 * t + (e & 1)] = o[i][e];
  if (t == 0) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      sm[warp * kHeads + gr + i * 8] = m[i];
      sl[warp * kHeads + gr + i * 8] = l[i];
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * D; i += kWarps * 32) {
    const int h = i / D, c = i - h * D;
    float mx = -INFINITY;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) mx = fmaxf(mx, sm[w * kHeads + h]);
    float den = 0.f, v = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float mw = sm[w * kHeads + h];
      if (mw == -INFINITY) continue;
      const float f = exp2f(mw - mx);
      den += f * sl[w * kHeads + h];
      v += f * so[(w * kHeads + h) * C::DP + c];
    }
    const long long oh = static_cast<long long>(b) * a.Hq + hq0 + h;
    if (n_splits == 1) {
      static_cast<bf16*>(a.out)[oh * D + c] = __float2bfloat16_rn(den > 0.f ? v / den : 0.f);
    } else {
      float* ws = a.ws + (oh * n_splits + split) * (D + 2);
      ws[c] = v;
      if (c == 0) {
        ws[D] = mx;
        ws[D + 1] = den;
      }
    }
  }
}

template <int KD>
const char* launch(const BiasDecodeArgs& a, int n_splits, cudaStream_t s) {
  auto k = bias_decode_tc_kernel<KD>;
  if (!FERRL_ONCE_PER_DEVICE(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<KD>::SMEM) == cudaSuccess))
    return "bias_decode: cannot reserve shared memory";
  const int rep = a.Hq / a.Hkv;
  launch_pdl(k, dim3(n_splits, a.Hkv * ((rep + kHeads - 1) / kHeads), a.B), dim3(kWarps * 32), Cfg<KD>::SMEM, s, a, n_splits);
  count_launch();
  return cudaGetLastError() == cudaSuccess ? nullptr : "bias_decode launch failed";
}

}  // namespace

bool bias_decode_tc_supported(const BiasDecodeArgs& a) {
  auto al = [](const void* p, unsigned n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  return a.dtype == kBF16 && a.D % 8 == 0 && a.D <= 256 && a.ld_k % 8 == 0 && a.ld_q % 2 == 0 && al(a.q, 4) && al(a.k, 16) && al(a.cache, 16);
}

// ranges of a row: enough CTAs for two waves of the device, at least two blocks of every warp each
int bias_decode_splits(const BiasDecodeArgs& a, int num_sms) {
  const int rep = a.Hq / a.Hkv, ctas = std::max(1, a.B * a.Hkv * ((rep + kHeads - 1) / kHeads));
  return std::max(1, std::min({2 * num_sms / ctas, a.slots / (2 * kKeys * kWarps), 32}));
}

const char* bias_decode_tc(const BiasDecodeArgs& a, int n_splits, cudaStream_t s) {
  if (!bias_decode_tc_supported(a)) return "bias_decode: unsupported arguments";
  if (a.B == 0) return nullptr;
  if (n_splits > 1 && !a.ws) return "bias_decode: workspace missing";
  const int kd = (a.D + 15) / 16;
  const char* err = kd <= 2 ? launch<2>(a, n_splits, s) : kd <= 4 ? launch<4>(a, n_splits, s) : kd <= 6 ? launch<6>(a, n_splits, s)
                  : kd <= 8 ? launch<8>(a, n_splits, s) : kd <= 12 ? launch<12>(a, n_splits, s) : launch<16>(a, n_splits, s);
  if (err || n_splits == 1) return err;
  return attn_combine(a.ws, nullptr, a.out, static_cast<long long>(a.B) * a.Hq, a.Hq, a.D, n_splits, s);
}

}  // namespace ferrl
