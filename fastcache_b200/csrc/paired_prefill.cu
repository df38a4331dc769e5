// Causal prefill attention on tcgen05 for keys that all heads share (LatentPrefill with D = 0, up to 256 columns): one CTA owns 128
// query rows of TWO heads of the same value head, so that every key and value tile is loaded once for both.
//
// Key tiles of 64 rows.  Scores are double-buffered, so that the next tile's products run while this one's softmax does:
//     S of head x, buffer b [(2 x + b) * 64, + 64)   O of head x [256 + 128 x, + 128)
//   warp 0       TMA: the Q tiles of both heads once, K in sub-tiles of 64 columns through a ring, V tiles in two stages
//   warp 1       tcgen05.mma issuer: for every K sub-tile both heads' scores, then the slot is free; O_x += P_x V with P_x in tensor
//                memory over S_x
//   warps 2-5    softmax of the first head, warps 6-9 of the second: one query row per thread, reference maximum as in
//                latent_prefill.cu
// Barriers of a score buffer are separate: a head's softmax may be a tile ahead of the other's.
#include <cuda.h>
#include <algorithm>
#include <stdexcept>
#include <string>

#include "gemm.h"
#include "hybrid.cuh"
#include "one_lane.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int PP_BM = 128, PP_BN = 64, PP_THREADS = 320;
constexpr int PP_QSUB = PP_BM * 128, PP_SUB = PP_BN * 128;      // bytes of a sub-tile of 64 columns: queries; keys or values
constexpr int PP_RING = 8;                                      // most slots of the K ring
constexpr int PP_BYTES = 224 * 1024;                            // Q, K ring, V
constexpr float PP_RESCALE = 8.f;                               // log2 units

__device__ __forceinline__ uint64_t pp_sdesc(uint32_t addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  uint64_t d = 0;
  d |= uint64_t((addr & 0x3FFFF) >> 4);
  d |= uint64_t((lbo_bytes >> 4) & 0x3FFF) << 16;
  d |= uint64_t((sbo_bytes >> 4) & 0x3FFF) << 32;
  d |= uint64_t(1) << 46;
  d |= uint64_t(2) << 61;
  return d;
}

struct PpMaps {
  CUtensorMap q, k, v;
};
struct PpParams {
  const int *cu_q, *cu_kv;
  bf16* out;
  long long ld_out;
  int R, V, heads_per_value, nq, ring;
  float scale_log2;
  uint32_t* status;
};

template <int NV>
__global__ void __launch_bounds__(PP_THREADS, 1)
paired_prefill_kernel(const __grid_constant__ PpMaps tm, const PpParams p) {
  constexpr int V_BYTES = NV * PP_SUB;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* s_q = smem;                             // [2 heads][nq]
  uint8_t* s_v = s_q + 2 * p.nq * PP_QSUB;         // [2 stages]
  uint8_t* s_k = s_v + 2 * V_BYTES;                // ring
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + PP_BYTES);
  uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = k_full + PP_RING, *v_full = k_empty + PP_RING, *v_empty = v_full + 2;
  uint64_t *s_full = v_empty + 2, *p_ready = s_full + 4, *o_done = p_ready + 4;     // [head][buffer], [head][buffer], [head]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 2);
  volatile int* s_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.z, h0 = blockIdx.y * 2;
  const int q_begin = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q_begin;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * PP_BM;            // late (long) tiles first
  if (q0 >= q_len) return;
  const int kv_begin = p.cu_kv[seq], kv_len = p.cu_kv[seq + 1] - kv_begin;
  const int offset = kv_len - q_len;
  const int kv_end = min(kv_len, offset + q0 + PP_BM);
  const int n_tiles = (kv_end + PP_BN - 1) / PP_BN;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < p.ring; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
      mbar_init(&o_done[s], 1);
    }
    for (int s = 0; s < 4; ++s) {
      mbar_init(&s_full[s], 1);
      mbar_init(&p_ready[s], 128);
    }
    *s_abort = 0;
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA loader
    const uint32_t el = elect_one() ? 1u : 0u;
    one_expect(q_full, uint32_t(2 * p.nq) * PP_QSUB, el);
    for (int i = 0; i < 2 * p.nq; ++i) {
      const int x = i >= p.nq ? 1 : 0;
      one_load_3d(s_q + i * PP_QSUB, &tm.q, q_full, (i - x * p.nq) * 64, h0 + x, q_begin + q0, el);
    }
    const int hv = h0 / p.heads_per_value;
    int slot = 0;
    uint32_t phase = 1;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int row = kv_begin + j * PP_BN;
      ok = !__any_sync(0xffffffffu, *s_abort != 0);
      for (int i = 0; i < p.nq && ok; ++i) {
        ok = warp_wait(&k_empty[slot], phase, p.status, ST_TIMEOUT_EMPTY);
        if (!ok) break;
        one_expect(&k_full[slot], PP_SUB, el);
        one_load_2d(s_k + slot * PP_SUB, &tm.k, &k_full[slot], i * 64, row, el);
        if (++slot == p.ring) {
          slot = 0;
          phase ^= 1;
        }
      }
      if (!ok) break;
      const int st = j & 1;
      ok = warp_wait(&v_empty[st], (uint32_t(j >> 1) & 1u) ^ 1u, p.status, ST_TIMEOUT_EMPTY);
      if (!ok) break;
      one_expect(&v_full[st], V_BYTES, el);
#pragma unroll
      for (int s = 0; s < NV; ++s) one_load_3d(s_v + st * V_BYTES + s * PP_SUB, &tm.v, &v_full[st], s * 64, hv, row, el);
    }
    if (!ok && lane == 0) *s_abort = 1;
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    const uint32_t el = elect_one() ? 1u : 0u;
    constexpr uint32_t idesc_s = make_idesc_bf16(128, PP_BN, false, false);
    constexpr uint32_t idesc_o = make_idesc_bf16(128, NV * 64, false, true);     // B (= V) is MN-major
    const uint64_t d_k = pp_sdesc(smem_u32(s_k), 16, 1024), d_q = pp_sdesc(smem_u32(s_q), 16, 1024);
    const uint64_t d_v = pp_sdesc(smem_u32(s_v), PP_SUB, 1024);
    int slot = 0;
    uint32_t phase = 0;
    auto issue_s = [&](int j) {
      const uint32_t ts = tmem + uint32_t(j & 1) * 64u;
      for (int i = 0; i < p.nq; ++i) {
        if (!warp_wait(&k_full[slot], phase, p.status, ST_TIMEOUT_FULL)) return false;
        tc_fence_after();
        const uint64_t dk = d_k + uint64_t(slot * (PP_SUB >> 4));
        const int left = p.R - i * 64;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const uint64_t dq = d_q + uint64_t((x * p.nq + i) * (PP_QSUB >> 4));
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            if (kk * 16 < left)
              one_mma(ts + uint32_t(x) * 128u, dq + uint64_t(kk * 2), dk + uint64_t(kk * 2), idesc_s, (i > 0 || kk > 0) ? 1u : 0u, el);
        }
        one_commit(&k_empty[slot], el);
        if (++slot == p.ring) {
          slot = 0;
          phase ^= 1;
        }
      }
      one_commit(&s_full[j & 1], el);
      one_commit(&s_full[2 + (j & 1)], el);
      return true;
    };
    bool ok = warp_wait(q_full, 0, p.status, ST_TIMEOUT_FULL) && issue_s(0);
    for (int j = 0; j < n_tiles && ok; ++j) {
      // the other buffer: its P went into O two products ago
      if (j + 1 < n_tiles) ok = issue_s(j + 1);
      const int b = j & 1;
      const uint32_t use = uint32_t(j >> 1) & 1u;
      ok = ok && warp_wait(&v_full[b], use, p.status, ST_TIMEOUT_FULL);
      const uint64_t dv = d_v + uint64_t(b * (V_BYTES >> 4));
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        ok = ok && warp_wait(&p_ready[2 * x + b], use, p.status, ST_TIMEOUT_FULL);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < PP_BN / 16; ++kk)
          one_mma_ts(tmem + 256u + uint32_t(x) * 128u, tmem + uint32_t(2 * x + b) * 64u + uint32_t(kk * 8), dv + uint64_t(kk * 128), idesc_o,
                     (j > 0 || kk > 0) ? 1u : 0u, el);
        one_commit(&o_done[x], el);
      }
      if (ok) one_commit(&v_empty[b], el);
    }
    if (!ok && lane == 0) *s_abort = 1;
  } else {
    // ------------------------------------------------ softmax and epilogue of one head
    const int x = (warp - 2) >> 2;
    const int lane_group = warp & 3;                         // TMEM lanes this warp may touch
    const int row = lane_group * 32 + lane;
    const uint32_t lanes = uint32_t(lane_group * 32) << 16;
    const uint32_t to = tmem + lanes + 256u + uint32_t(x * 128);
    const int qrow = q0 + row, qpos = offset + qrow;
    float m_ref = -INFINITY, l = 0.f;                        // -inf: no visible key yet
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int b = 2 * x + (j & 1);
      const uint32_t ts = tmem + lanes + uint32_t(b * 64);
      if (!__all_sync(0xffffffffu, !*s_abort && mbar_wait(&s_full[b], uint32_t(j >> 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL))) {
        ok = false;
        break;
      }
      tc_fence_after();
      uint32_t s[64];
      tmem_ld_32x32(ts, *reinterpret_cast<uint32_t(*)[32]>(&s[0]));
      tmem_ld_32x32(ts + 32u, *reinterpret_cast<uint32_t(*)[32]>(&s[32]));
      tmem_ld_wait();
      const int col0 = j * PP_BN;
      if (col0 + PP_BN - 1 > offset + q0 || col0 + PP_BN > kv_end) {
        const int last = min(qpos, kv_end - 1) - col0;
#pragma unroll
        for (int t = 0; t < PP_BN; ++t)
          if (t > last) s[t] = 0xff800000u;                  // -inf
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int t = 0; t < PP_BN; ++t) mx4[t & 3] = fmaxf(mx4[t & 3], __uint_as_float(s[t]));
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2;
      if (j == 0) {
        m_ref = mx;
      } else if (__any_sync(0xffffffffu, mx > m_ref + PP_RESCALE)) {
        // some row of this warp outgrew its reference: bring O_x (complete up to the tile before) to the new one
        if (!__all_sync(0xffffffffu, mbar_wait(&o_done[x], uint32_t(j - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL))) {
          ok = false;
          break;
        }
        tc_fence_after();
        const float m_new = fmaxf(m_ref, mx);
        const float f = m_ref == -INFINITY ? 0.f : exp2f(m_ref - m_new);
        m_ref = m_new;
        l *= f;
#pragma unroll 1
        for (int c = 0; c < NV * 2; ++c) {
          uint32_t r[32];
          tmem_ld_32x32(to + uint32_t(c * 32), r);
          tmem_ld_wait();
#pragma unroll
          for (int t = 0; t < 32; ++t) r[t] = __float_as_uint(__uint_as_float(r[t]) * f);
          tmem_st_32x32(to + uint32_t(c * 32), r);
        }
        tmem_st_wait();
      }
      const float base = m_ref == -INFINITY ? 0.f : m_ref;
      float rs[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t u[32];
#pragma unroll
      for (int t = 0; t < 32; ++t) {
        float e0, e1;
        const float a0 = fmaf(__uint_as_float(s[2 * t]), p.scale_log2, -base);
        const float a1 = fmaf(__uint_as_float(s[2 * t + 1]), p.scale_log2, -base);
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e0) : "f"(a0));
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e1) : "f"(a1));
        rs[t & 3] += e0 + e1;
        u[t] = pack_bf16(e0, e1);
      }
      tmem_st_32x32(ts, u);
      tmem_st_wait();
      l += (rs[0] + rs[1]) + (rs[2] + rs[3]);
      // the last two phases of o_done one by one, a parity cannot tell a phase from the one two before it: the scores of the last
      // tile only say that the third-last product is done, and the last one cannot be before this arrival
      if (j == n_tiles - 1 && j > 0) ok = mbar_wait(&o_done[x], uint32_t(j - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL);
      tc_fence_before();
      mbar_arrive(&p_ready[b]);
    }
    if (ok) ok = mbar_wait(&o_done[x], uint32_t(n_tiles - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL);
    if (!ok) *s_abort = 1;
    tc_fence_after();
    if (__all_sync(0xffffffffu, ok)) {
      const float inv = l > 0.f ? 1.f / l : 0.f;
      bf16* dst = p.out + (long long)(q_begin + qrow) * p.ld_out + (h0 + x) * p.V;
#pragma unroll 1
      for (int c = 0; c < NV * 2; ++c) {
        uint32_t r[32];
        tmem_ld_32x32(to + uint32_t(c * 32), r);
        tmem_ld_wait();
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int col = c * 32 + q * 8;
          if (qrow >= q_len || col >= p.V) continue;         // V is a multiple of 8
          uint32_t ow[4];
#pragma unroll
          for (int e = 0; e < 4; ++e)
            ow[e] = pack_bf16(__uint_as_float(r[q * 8 + 2 * e]) * inv, __uint_as_float(r[q * 8 + 2 * e + 1]) * inv);
          *reinterpret_cast<uint4*>(dst + col) = make_uint4(ow[0], ow[1], ow[2], ow[3]);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

bool paired_prefill_supported(const LatentPrefill& p) {
  return latent_prefill_supported(p) && p.D == 0 && p.R <= 256 && p.window == 0 && p.sink == nullptr && p.gate == nullptr &&
         p.head_gate == nullptr && p.v_heads > 0 && (p.H / p.v_heads) % 2 == 0;
}

void launch_paired_prefill(const LatentPrefill& p, cudaStream_t s) {
  if (p.T == 0 || p.B == 0 || p.max_q == 0) return;
  PpMaps tm;
  tm.q = make_tmap_bf16_3d(p.q, p.R, p.H, p.T, p.R, p.ld_q, 64, 1, PP_BM);
  tm.k = make_tmap_bf16_2d(p.rot, p.total_kv, p.R, p.ld_rot, PP_BN, 64);
  tm.v = make_tmap_bf16_3d(p.v, p.V, p.v_heads, p.total_kv, p.V, p.ld_v, 64, 1, PP_BN);
  PpParams a;
  a.cu_q = p.cu_q;
  a.cu_kv = p.cu_kv;
  a.out = reinterpret_cast<bf16*>(p.out);
  a.ld_out = p.ld_out;
  a.R = p.R;
  a.V = p.V;
  a.heads_per_value = p.H / p.v_heads;
  a.scale_log2 = p.scale * 1.4426950408889634f;
  a.status = p.status;
  a.nq = (p.R + 63) / 64;
  const int nv = p.V <= 64 ? 1 : 2;
  a.ring = std::min(PP_RING, (PP_BYTES - 2 * a.nq * PP_QSUB - 2 * nv * PP_SUB) / PP_SUB);
  // barriers behind the tiles, then the slack of the alignment
  constexpr int smem = PP_BYTES + (2 * PP_RING + 18) * 8 + 1024;
  static_assert(smem <= 227 * 1024, "shared memory of a CTA");
  auto go = [&](auto kern) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    kern<<<dim3((p.max_q + PP_BM - 1) / PP_BM, p.H / 2, p.B), PP_THREADS, smem, s>>>(tm, a);
  };
  if (nv == 1) go(paired_prefill_kernel<1>);
  else go(paired_prefill_kernel<2>);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("prefill of paired heads: ") + cudaGetErrorString(e));
}

}  // namespace fc
