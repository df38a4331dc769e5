// Causal prefill attention on tcgen05 over the gathered cache rows of each request (contiguous, see launch_gather_rows): keys
// of D columns per head and R columns that all heads share, values of another size.  Latent attention: D and values expanded
// from the rows, R the rotated part.  Heads that mix their scores: D = 0, R the keys of all key heads side by side, values of
// a group of heads.  Options: sliding window (key tiles before a query tile's window are neither loaded nor multiplied), sink.
//
// One CTA owns 128 query rows of one head and walks the visible keys in tiles of 128.  Even and odd key tiles have
// separate score and output accumulators in tensor memory and separate softmax warps, so that one parity's matrices
// run while the other's softmax does; the two partial results are merged at the end:
//     S_0 [0,128)  S_1 [128,256)  O_0 [256,384)  O_1 [384,512)
//   warp 0       TMA: the Q tile once, K through a ring whose slots take one or more sub-tiles of 64 columns (a whole tile
//                where two fit), V tiles.  Queries of more than eight sub-tiles do not stay: every slot then takes a sub-tile
//                of K and of Q.  Three-dimensional boxes (column, head, row) zero-fill the columns past a head's width
//   warp 1       tcgen05.mma issuer: S_x = Q K(j)^T, then O_x += P_x V(j) with P_x in tensor memory over S_x
//   warps 2-5    softmax of even tiles, warps 6-9 of odd tiles: one query row per thread, reference maximum as in
//                attn_prefill_tc2.cu (O is rescaled only when a row outgrows its reference by 2^8)
// The epilogue multiplies with the output gate, if there is one, and writes bf16.
#include <cuda.h>
#include <algorithm>
#include <stdexcept>
#include <string>

#include "gemm.h"
#include "hybrid.cuh"
#include "one_lane.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int LP_BM = 128, LP_BN = 128, LP_THREADS = 320;
constexpr int LP_SUB = 128 * 128;                 // bytes of a [128 rows x 64 columns] sub-tile
constexpr float LP_RESCALE = 8.f;                 // log2 units
constexpr int LP_SLOTS = 14;                      // sub-tiles of shared memory: Q, K ring, V
constexpr int LP_RING = 8;                        // most slots of the K ring
constexpr float LP_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ uint64_t lp_sdesc(uint32_t addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  uint64_t d = 0;
  d |= uint64_t((addr & 0x3FFFF) >> 4);
  d |= uint64_t((lbo_bytes >> 4) & 0x3FFF) << 16;
  d |= uint64_t((sbo_bytes >> 4) & 0x3FFF) << 32;
  d |= uint64_t(1) << 46;
  d |= uint64_t(2) << 61;
  return d;
}

struct LpMaps {
  CUtensorMap qn, qr, kn, kr, v;
};
struct LpParams {
  const int *cu_q, *cu_kv;
  const bf16* gate;
  const float *head_gate, *sink;
  bf16* out;
  long long ld_gate, ld_out;
  int D, R, V, heads_per_value, window;
  int nd, nr;                                     // sub-tiles of the keys' own and shared columns
  int ring, per_slot, v_stages;                   // slots of the K ring, sub-tiles of K in a slot
  float scale_log2;
  uint32_t* status;
};

// NV: 64-column sub-tiles of the values; STREAM_Q: Q comes with K through the ring
template <int NV, bool STREAM_Q>
__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ LpMaps tm, const LpParams p) {
  const int slot_bytes = STREAM_Q ? 2 * LP_SUB : p.per_slot * LP_SUB;    // STREAM_Q: K sub-tile, then Q's
  constexpr int V_BYTES = NV * LP_SUB;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nq = p.nd + p.nr;                      // sub-tiles of a Q or K tile
  uint8_t* s_k = smem;                             // ring
  uint8_t* s_v = s_k + p.ring * slot_bytes;              // v_stages
  uint8_t* s_q = s_v + p.v_stages * V_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + LP_SLOTS * LP_SUB);
  uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = k_full + LP_RING, *v_full = k_empty + LP_RING, *v_empty = v_full + 2;
  uint64_t *s_full = v_empty + 2, *p_ready = s_full + 2, *o_done = p_ready + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 2);
  volatile int* s_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_ml = reinterpret_cast<float*>(o_done + 3);   // [2][128] reference maximum and sum of the odd tiles

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.z, h = blockIdx.x;
  const int q_begin = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q_begin;
  const int q0 = (gridDim.y - 1 - blockIdx.y) * LP_BM;            // late (long) tiles first
  if (q0 >= q_len) return;
  const int kv_begin = p.cu_kv[seq], kv_len = p.cu_kv[seq + 1] - kv_begin;
  const int offset = kv_len - q_len;
  const int kv_end = min(kv_len, offset + q0 + LP_BM);
  const int first_key = p.window > 0 ? max(0, offset + q0 - p.window + 1) : 0;      // of the tile's first row
  const int tile0 = first_key / LP_BN;
  const int n_tiles = (kv_end + LP_BN - 1) / LP_BN - tile0;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < p.ring; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
      mbar_init(&s_full[s], 1);
      mbar_init(&p_ready[s], 128);
      mbar_init(&o_done[s], 1);
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
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA loader
    const uint32_t el = elect_one() ? 1u : 0u;
    auto load_q = [&](uint8_t* dst, uint64_t* bar, int i) {
      if (i < p.nd) one_load_3d(dst, &tm.qn, bar, i * 64, h, q_begin + q0, el);
      else one_load_3d(dst, &tm.qr, bar, (i - p.nd) * 64, h, q_begin + q0, el);
    };
    if (!STREAM_Q) {
      one_expect(q_full, uint32_t(nq) * LP_SUB, el);
      for (int i = 0; i < nq; ++i) load_q(s_q + i * LP_SUB, q_full, i);
    }
    const int hv = h / p.heads_per_value;
    int slot = 0;
    uint32_t phase = 1;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int row = kv_begin + (tile0 + j) * LP_BN;
      ok = !__any_sync(0xffffffffu, *s_abort != 0);
      for (int i0 = 0; i0 < nq && ok; i0 += p.per_slot) {
        ok = warp_wait(&k_empty[slot], phase, p.status, ST_TIMEOUT_EMPTY);
        if (!ok) break;
        uint8_t* dk = s_k + slot * slot_bytes;
        one_expect(&k_full[slot], slot_bytes, el);
        for (int i = i0; i < i0 + p.per_slot; ++i, dk += LP_SUB)
          if (i < p.nd) one_load_3d(dk, &tm.kn, &k_full[slot], i * 64, h, row, el);
          else one_load_2d(dk, &tm.kr, &k_full[slot], (i - p.nd) * 64, row, el);
        if (STREAM_Q) load_q(dk, &k_full[slot], i0);
        if (++slot == p.ring) {
          slot = 0;
          phase ^= 1;
        }
      }
      if (!ok) break;
      const int st = p.v_stages == 2 ? j & 1 : 0;
      const uint32_t use = uint32_t(p.v_stages == 2 ? j >> 1 : j) & 1u;
      ok = warp_wait(&v_empty[st], use ^ 1u, p.status, ST_TIMEOUT_EMPTY);
      if (!ok) break;
      one_expect(&v_full[st], V_BYTES, el);
#pragma unroll
      for (int s = 0; s < NV; ++s) one_load_3d(s_v + st * V_BYTES + s * LP_SUB, &tm.v, &v_full[st], s * 64, hv, row, el);
    }
    if (!ok && lane == 0) *s_abort = 1;
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    const uint32_t el = elect_one() ? 1u : 0u;
    constexpr uint32_t idesc_s = make_idesc_bf16(128, 128, false, false);
    constexpr uint32_t idesc_o = make_idesc_bf16(128, NV * 64, false, true);     // B (= V) is MN-major
    // descriptors by addition on their address field (16-byte units)
    const uint64_t d_k = lp_sdesc(smem_u32(s_k), 16, 1024), d_q = lp_sdesc(smem_u32(s_q), 16, 1024);
    const uint64_t d_v = lp_sdesc(smem_u32(s_v), LP_SUB, 1024);
    int slot = 0;
    uint32_t phase = 0;
    auto issue_s = [&](int j) {
      const uint32_t ts = tmem_base + uint32_t(j & 1) * 128u;
      for (int i0 = 0; i0 < nq; i0 += p.per_slot) {
        if (!warp_wait(&k_full[slot], phase, p.status, ST_TIMEOUT_FULL)) return false;
        tc_fence_after();
        uint64_t dk = d_k + uint64_t(slot * (slot_bytes >> 4)), dq = STREAM_Q ? dk + uint64_t(LP_SUB >> 4) : d_q + uint64_t(i0 * (LP_SUB >> 4));
        for (int i = i0; i < i0 + p.per_slot; ++i, dk += uint64_t(LP_SUB >> 4), dq += uint64_t(LP_SUB >> 4)) {
          const int left = i < p.nd ? p.D - i * 64 : p.R - (i - p.nd) * 64;
          if (elect_one())
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              if (kk * 16 < left)
                tc_mma_f16(ts, dq + uint64_t(kk * 2), dk + uint64_t(kk * 2), idesc_s, (i > 0 || kk > 0) ? 1u : 0u);
          __syncwarp();
        }
        one_commit(&k_empty[slot], el);
        if (++slot == p.ring) {
          slot = 0;
          phase ^= 1;
        }
      }
      one_commit(&s_full[j & 1], el);
      return true;
    };
    bool ok = STREAM_Q || warp_wait(q_full, 0, p.status, ST_TIMEOUT_FULL);
    if (ok) ok = issue_s(0);
    if (ok && n_tiles > 1) ok = issue_s(1);
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int x = j & 1, st = p.v_stages == 2 ? x : 0;
      ok = warp_wait(&p_ready[x], uint32_t(j >> 1) & 1u, p.status, ST_TIMEOUT_FULL) &&
           warp_wait(&v_full[st], uint32_t(p.v_stages == 2 ? j >> 1 : j) & 1u, p.status, ST_TIMEOUT_FULL);
      if (!ok) break;
      tc_fence_after();
      const uint64_t dv = d_v + uint64_t(st * (V_BYTES >> 4));
      if (elect_one())
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          tc_mma_f16_ts(tmem_base + 256u + uint32_t(x * 128), tmem_base + uint32_t(x * 128) + uint32_t(kk * 8), dv + uint64_t(kk * 128),
                        idesc_o, (j > 1 || kk > 0) ? 1u : 0u);
      __syncwarp();
      one_commit(&o_done[x], el);
      one_commit(&v_empty[st], el);
      if (j + 2 < n_tiles) ok = issue_s(j + 2);
    }
    if (!ok && lane == 0) *s_abort = 1;
  } else {
    // ------------------------------------------------ softmax of the even (x = 0) or odd (x = 1) key tiles
    const int x = (warp - 2) >> 2;
    const int lane_group = warp & 3;                         // TMEM lanes this warp may touch
    const int row = lane_group * 32 + lane;
    const uint32_t lane_addr = uint32_t(lane_group * 32) << 16;
    const uint32_t ts = tmem_base + lane_addr + uint32_t(x * 128);           // S_x, then P_x
    const uint32_t to = tmem_base + lane_addr + 256u + uint32_t(x * 128);    // O_x
    const int qrow = q0 + row;
    const int qpos = offset + qrow;
    const int n_x = (n_tiles + 1 - x) / 2;
    float m_ref = -INFINITY, l = 0.f;                        // -inf: no visible key yet
    bool ok = true;
    for (int i = 0; i < n_x && ok; ++i) {
      const int j = 2 * i + x;
      if (*s_abort || !mbar_wait(&s_full[x], uint32_t(i) & 1u, p.status, ST_TIMEOUT_ACC_FULL)) {
        ok = false;
        break;
      }
      tc_fence_after();
      uint32_t s[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32(ts + uint32_t(c * 32), *reinterpret_cast<uint32_t(*)[32]>(&s[c * 32]));
      tmem_ld_wait();
      const int col0 = (tile0 + j) * LP_BN;
      if ((col0 + LP_BN - 1 > offset + q0) || (col0 + LP_BN > kv_end)) {
#pragma unroll
        for (int t = 0; t < 128; ++t) {
          const int col = col0 + t;
          if (col > qpos || col >= kv_end) s[t] = 0xff800000u;          // -inf
        }
      }
      if (p.window > 0 && col0 <= offset + q0 + LP_BM - 1 - p.window) {  // the last row's window starts behind col0
        const int hidden = qpos - p.window - col0;
#pragma unroll
        for (int t = 0; t < 128; ++t)
          if (t <= hidden) s[t] = 0xff800000u;
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};        // four chains
#pragma unroll
      for (int t = 0; t < 128; ++t) mx4[t & 3] = fmaxf(mx4[t & 3], __uint_as_float(s[t]));
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2;
      if (i == 0) {
        m_ref = mx;
      } else if (__any_sync(__activemask(), mx > m_ref + LP_RESCALE)) {
        // some row of this warp outgrew its reference: bring O_x (complete up to the tile before) to the new one
        if (!mbar_wait(&o_done[x], uint32_t(i - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL)) {
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
      uint32_t u[64];
#pragma unroll
      for (int t = 0; t < 64; ++t) {
        float e0, e1;
        const float a0 = fmaf(__uint_as_float(s[2 * t]), p.scale_log2, -base);
        const float a1 = fmaf(__uint_as_float(s[2 * t + 1]), p.scale_log2, -base);
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e0) : "f"(a0));
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e1) : "f"(a1));
        rs[t & 3] += e0 + e1;
        u[t] = pack_bf16(e0, e1);
      }
      tmem_st_32x32(ts, *reinterpret_cast<uint32_t(*)[32]>(&u[0]));
      tmem_st_32x32(ts + 32u, *reinterpret_cast<uint32_t(*)[32]>(&u[32]));
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_ready[x]);
      l += (rs[0] + rs[1]) + (rs[2] + rs[3]);
    }
    if (ok && n_x > 0) ok = mbar_wait(&o_done[x], uint32_t(n_x - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL);
    if (!ok) *s_abort = 1;
    tc_fence_after();
    // every matrix of both parities is done after this barrier: the K stages are free for the odd tiles' result
    asm volatile("bar.sync 1, 256;" ::: "memory");
    float* s_o = reinterpret_cast<float*>(s_k);                  // [NV * 64 columns][128 rows]: two slots per 64 columns
    const bool two = n_tiles > 1 && !*s_abort;
    if (x == 1) {
      if (two) {
        s_ml[row] = m_ref;
        s_ml[128 + row] = l;
#pragma unroll 1
        for (int c = 0; c < NV * 2; ++c) {
          uint32_t r[32];
          tmem_ld_32x32(to + uint32_t(c * 32), r);
          tmem_ld_wait();
#pragma unroll
          for (int t = 0; t < 32; ++t) s_o[(c * 32 + t) * 128 + row] = __uint_as_float(r[t]);
        }
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");
    } else {
      asm volatile("bar.sync 1, 256;" ::: "memory");
      if (ok) {
        float w0 = 1.f, w1 = 0.f, mm = m_ref;                    // a row sees itself: one of the maxima is finite
        if (two) {
          const float m1 = s_ml[row];
          mm = fmaxf(m_ref, m1);
          w0 = m_ref == -INFINITY ? 0.f : exp2f(m_ref - mm);
          w1 = m1 == -INFINITY ? 0.f : exp2f(m1 - mm);
          l = l * w0 + s_ml[128 + row] * w1;
        }
        if (p.sink != nullptr && l > 0.f) l += exp2f(p.sink[h] * LP_LOG2E - mm);
        float inv = l > 0.f ? 1.f / l : 0.f;
        if (p.head_gate != nullptr && qrow < q_len) inv *= p.head_gate[(long long)(q_begin + qrow) * gridDim.x + h];
        w0 *= inv;
        w1 *= inv;
        bf16* dst = p.out + (long long)(q_begin + qrow) * p.ld_out + h * p.V;
        const bf16* gate = p.gate != nullptr ? p.gate + (long long)(q_begin + qrow) * p.ld_gate + h * p.V : nullptr;
#pragma unroll 1
        for (int c = 0; c < NV * 2; ++c) {
          uint32_t r[32];
          tmem_ld_32x32(to + uint32_t(c * 32), r);
          tmem_ld_wait();
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int col = c * 32 + q * 8;
            if (qrow >= q_len || col >= p.V) continue;           // V is a multiple of 8
            const uint4 gu = gate != nullptr ? *reinterpret_cast<const uint4*>(gate + col) : make_uint4(0, 0, 0, 0);
            const uint32_t gw[4] = {gu.x, gu.y, gu.z, gu.w};
            uint32_t ow[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float a = __uint_as_float(r[q * 8 + 2 * e]) * w0, b = __uint_as_float(r[q * 8 + 2 * e + 1]) * w0;
              if (two) {
                a = fmaf(s_o[(col + 2 * e) * 128 + row], w1, a);
                b = fmaf(s_o[(col + 2 * e + 1) * 128 + row], w1, b);
              }
              if (gate != nullptr) {
                const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[e]));
                a *= sigmoid_t<bf16>(g.x);
                b *= sigmoid_t<bf16>(g.y);
              }
              ow[e] = pack_bf16(a, b);
            }
            *reinterpret_cast<uint4*>(dst + col) = make_uint4(ow[0], ow[1], ow[2], ow[3]);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

bool latent_prefill_supported(const LatentPrefill& p) {
  return p.D % 8 == 0 && p.D <= 128 && p.R % 8 == 0 && p.V % 8 == 0 && p.V <= 128 && p.R > 0 && p.V > 0 && p.D >= 0 &&
         (p.v_heads == 0 || p.H % p.v_heads == 0);
}

template <int NV, bool STREAM_Q>
static void launch_lp(const LpMaps& tm, const LpParams& q, const LatentPrefill& p, cudaStream_t s) {
  // barriers and maxima behind the sub-tiles, then the slack of the alignment
  constexpr int smem = LP_SLOTS * LP_SUB + (2 * LP_RING + 14) * 8 + 1024 + 1024;
  static_assert(smem <= 227 * 1024, "shared memory of a CTA");
  auto kern = latent_prefill_kernel<NV, STREAM_Q>;
  cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  kern<<<dim3(p.H, (p.max_q + LP_BM - 1) / LP_BM, p.B), LP_THREADS, smem, s>>>(tm, q);
}

void launch_latent_prefill(const LatentPrefill& p, cudaStream_t s) {
  if (p.T == 0 || p.B == 0 || p.max_q == 0) return;
  LpMaps tm;
  const uint64_t Q = uint64_t(p.D + p.R);
  const int vh = p.v_heads > 0 ? p.v_heads : p.H;
  const bf16* q = reinterpret_cast<const bf16*>(p.q);
  tm.qr = make_tmap_bf16_3d(q + p.D, p.R, p.H, p.T, Q, p.ld_q, 64, 1, LP_BM);
  tm.kr = make_tmap_bf16_2d(p.rot, p.total_kv, p.R, p.ld_rot, LP_BN, 64);
  tm.qn = p.D > 0 ? make_tmap_bf16_3d(q, p.D, p.H, p.T, Q, p.ld_q, 64, 1, LP_BM) : tm.qr;
  tm.kn = p.D > 0 ? make_tmap_bf16_3d(p.k, p.D, p.H, p.total_kv, p.D, p.ld_k, 64, 1, LP_BN) : tm.kr;
  tm.v = make_tmap_bf16_3d(p.v, p.V, vh, p.total_kv, p.V, p.ld_v, 64, 1, LP_BN);
  LpParams a;
  a.cu_q = p.cu_q;
  a.cu_kv = p.cu_kv;
  a.gate = reinterpret_cast<const bf16*>(p.gate);
  a.head_gate = p.head_gate;
  a.sink = p.sink;
  a.out = reinterpret_cast<bf16*>(p.out);
  a.ld_gate = p.ld_gate;
  a.ld_out = p.ld_out;
  a.D = p.D;
  a.R = p.R;
  a.V = p.V;
  a.heads_per_value = p.H / vh;
  a.window = p.window;
  a.scale_log2 = p.scale * LP_LOG2E;
  a.status = p.status;
  a.nd = (p.D + 63) / 64;
  a.nr = (p.R + 63) / 64;
  const int nv = p.V <= 64 ? 1 : 2, nq = a.nd + a.nr;
  const bool stream = nq > 8;
  // at least four slots for K; two stages of V where they leave that much
  const int left = LP_SLOTS - (stream ? 0 : nq);
  a.v_stages = left - 2 * nv >= (stream ? 8 : 4) ? 2 : 1;
  const int subs = left - a.v_stages * nv;                 // of the ring
  a.per_slot = stream ? 1 : 2 * nq <= subs ? nq : nq % 2 == 0 ? 2 : 1;
  a.ring = std::min(LP_RING, subs / (stream ? 2 : a.per_slot));
  if (nv == 1) stream ? launch_lp<1, true>(tm, a, p, s) : launch_lp<1, false>(tm, a, p, s);
  else stream ? launch_lp<2, true>(tm, a, p, s) : launch_lp<2, false>(tm, a, p, s);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("prefill over gathered rows: ") + cudaGetErrorString(e));
}

}  // namespace fc
