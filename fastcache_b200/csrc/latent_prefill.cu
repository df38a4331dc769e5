// Causal prefill attention of latent layers on tcgen05: per-head keys and values expanded from the cache rows of each
// request (contiguous, see launch_gather_rows), key = [dim unrotated | rot shared by all heads], value of another size.
//
// One CTA owns 128 query rows of one head and walks the visible keys in tiles of 128.  Even and odd key tiles have
// separate score and output accumulators in tensor memory and separate softmax warps, so that one parity's matrices
// run while the other's softmax does; the two partial results are merged at the end:
//     S_0 [0,128)  S_1 [128,256)  O_0 [256,384)  O_1 [384,512)
//   warp 0       TMA: the Q tile once, then K (unrotated sub-tiles + rotated sub-tile) and V tiles; stage = parity.
//                Three-dimensional boxes (column, head, row) zero-fill the columns past a head's width
//   warp 1       tcgen05.mma issuer: S_x = Q K(j)^T, then O_x += P_x V(j) with P_x in tensor memory over S_x
//   warps 2-5    softmax of even tiles, warps 6-9 of odd tiles: one query row per thread, reference maximum as in
//                attn_prefill_tc2.cu (O is rescaled only when a row outgrows its reference by 2^8)
// The epilogue multiplies with sigmoid(gate) and writes bf16.
#include <cuda.h>
#include <stdexcept>
#include <string>

#include "gemm.h"
#include "hybrid.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int LP_BM = 128, LP_BN = 128, LP_THREADS = 320;
constexpr int LP_SUB = 128 * 128;                 // bytes of a [128 rows x 64 columns] sub-tile
constexpr float LP_RESCALE = 8.f;                 // log2 units

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
  bf16* out;
  long long ld_gate, ld_out;
  int D, R, V;
  float scale_log2;
  uint32_t* status;
};

// ND / NV: 64-column sub-tiles of the unrotated key part and of the values
template <int ND, int NV>
__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ LpMaps tm, const LpParams p) {
  constexpr int NQ = ND + 1;                       // sub-tiles of a Q or K tile: unrotated, then rotated
  constexpr int K_BYTES = NQ * LP_SUB, V_BYTES = NV * LP_SUB;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* s_q = smem;
  uint8_t* s_k = s_q + K_BYTES;                    // 2 stages
  uint8_t* s_v = s_k + 2 * K_BYTES;                // 2 stages
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_v + 2 * V_BYTES);
  uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = bars + 3, *v_full = bars + 5, *v_empty = bars + 7;
  uint64_t *s_full = bars + 9, *p_ready = bars + 11, *o_done = bars + 13;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* s_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_ml = reinterpret_cast<float*>(bars + 16);   // [2][128] reference maximum and sum of the odd tiles

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.z, h = blockIdx.y;
  const int q_begin = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q_begin;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * LP_BM;            // late (long) tiles first
  if (q0 >= q_len) return;
  const int kv_begin = p.cu_kv[seq], kv_len = p.cu_kv[seq + 1] - kv_begin;
  const int offset = kv_len - q_len;
  const int kv_end = min(kv_len, offset + q0 + LP_BM);
  const int n_tiles = (kv_end + LP_BN - 1) / LP_BN;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
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
    if (lane == 0) {
      mbar_expect_tx(q_full, K_BYTES);
#pragma unroll
      for (int s = 0; s < ND; ++s) tma_load_3d(s_q + s * LP_SUB, &tm.qn, q_full, s * 64, h, q_begin + q0);
      tma_load_3d(s_q + ND * LP_SUB, &tm.qr, q_full, 0, h, q_begin + q0);
      for (int j = 0; j < n_tiles && !*s_abort; ++j) {
        const int st = j & 1;
        const uint32_t ph = ((j >> 1) & 1) ^ 1;
        const int row = kv_begin + j * LP_BN;
        if (!mbar_wait(&k_empty[st], ph, p.status, ST_TIMEOUT_EMPTY)) {
          *s_abort = 1;
          break;
        }
        mbar_expect_tx(&k_full[st], K_BYTES);
        uint8_t* dk = s_k + st * K_BYTES;
#pragma unroll
        for (int s = 0; s < ND; ++s) tma_load_3d(dk + s * LP_SUB, &tm.kn, &k_full[st], s * 64, h, row);
        tma_load_2d(dk + ND * LP_SUB, &tm.kr, &k_full[st], 0, row);
        if (!mbar_wait(&v_empty[st], ph, p.status, ST_TIMEOUT_EMPTY)) {
          *s_abort = 1;
          break;
        }
        mbar_expect_tx(&v_full[st], V_BYTES);
#pragma unroll
        for (int s = 0; s < NV; ++s) tma_load_3d(s_v + st * V_BYTES + s * LP_SUB, &tm.v, &v_full[st], s * 64, h, row);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc_bf16(128, 128, false, false);
      constexpr uint32_t idesc_o = make_idesc_bf16(128, NV * 64, false, true);     // B (= V) is MN-major
      const int steps_d = (p.D + 15) / 16, steps_r = (p.R + 15) / 16;
      auto issue_s = [&](int j) {
        const int x = j & 1;
        if (!mbar_wait(&k_full[x], uint32_t(j >> 1) & 1u, p.status, ST_TIMEOUT_FULL)) return false;
        tc_fence_after();
        const uint32_t qa = smem_u32(s_q), ka = smem_u32(s_k + x * K_BYTES);
        for (int kk = 0; kk < steps_d; ++kk) {
          const uint32_t off = uint32_t(kk >> 2) * LP_SUB + uint32_t(kk & 3) * 32;
          tc_mma_f16(tmem_base + uint32_t(x * 128), lp_sdesc(qa + off, 16, 1024), lp_sdesc(ka + off, 16, 1024), idesc_s,
                     kk > 0 ? 1u : 0u);
        }
        for (int kk = 0; kk < steps_r; ++kk) {
          const uint32_t off = uint32_t(ND) * LP_SUB + uint32_t(kk) * 32;
          tc_mma_f16(tmem_base + uint32_t(x * 128), lp_sdesc(qa + off, 16, 1024), lp_sdesc(ka + off, 16, 1024), idesc_s,
                     1u);
        }
        tc_commit(&s_full[x]);
        tc_commit(&k_empty[x]);
        return true;
      };
      bool ok = mbar_wait(q_full, 0, p.status, ST_TIMEOUT_FULL);
      if (ok) ok = issue_s(0);
      if (ok && n_tiles > 1) ok = issue_s(1);
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int x = j & 1;
        const uint32_t use = uint32_t(j >> 1) & 1u;
        ok = mbar_wait(&p_ready[x], use, p.status, ST_TIMEOUT_FULL) &&
             mbar_wait(&v_full[x], use, p.status, ST_TIMEOUT_FULL);
        if (!ok) break;
        tc_fence_after();
        const uint32_t va = smem_u32(s_v + x * V_BYTES);
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          tc_mma_f16_ts(tmem_base + 256u + uint32_t(x * 128), tmem_base + uint32_t(x * 128) + uint32_t(kk * 8),
                        lp_sdesc(va + uint32_t(kk) * 2048, LP_SUB, 1024), idesc_o, (j > 1 || kk > 0) ? 1u : 0u);
        tc_commit(&o_done[x]);
        tc_commit(&v_empty[x]);
        if (j + 2 < n_tiles) ok = issue_s(j + 2);
      }
      if (!ok) *s_abort = 1;
    }
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
      const int col0 = j * LP_BN;
      if ((col0 + LP_BN - 1 > offset + q0) || (col0 + LP_BN > kv_end)) {
#pragma unroll
        for (int t = 0; t < 128; ++t) {
          const int col = col0 + t;
          if (col > qpos || col >= kv_end) s[t] = 0xff800000u;          // -inf
        }
      }
      float mx = -INFINITY;
#pragma unroll
      for (int t = 0; t < 128; ++t) mx = fmaxf(mx, __uint_as_float(s[t]));
      mx *= p.scale_log2;
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
      float rs = 0.f;
      uint32_t u[64];
#pragma unroll
      for (int t = 0; t < 64; ++t) {
        float e0, e1;
        const float a0 = fmaf(__uint_as_float(s[2 * t]), p.scale_log2, -base);
        const float a1 = fmaf(__uint_as_float(s[2 * t + 1]), p.scale_log2, -base);
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e0) : "f"(a0));
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e1) : "f"(a1));
        rs += e0 + e1;
        u[t] = pack_bf16(e0, e1);
      }
      tmem_st_32x32(ts, *reinterpret_cast<uint32_t(*)[32]>(&u[0]));
      tmem_st_32x32(ts + 32u, *reinterpret_cast<uint32_t(*)[32]>(&u[32]));
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_ready[x]);
      l += rs;
    }
    if (ok && n_x > 0) ok = mbar_wait(&o_done[x], uint32_t(n_x - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL);
    if (!ok) *s_abort = 1;
    tc_fence_after();
    // every matrix of both parities is done after this barrier: the K stages are free for the odd tiles' result
    asm volatile("bar.sync 1, 256;" ::: "memory");
    float* s_o = reinterpret_cast<float*>(s_k);                  // [NV * 64 columns][128 rows]
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
        float w0 = 1.f, w1 = 0.f;
        if (two) {
          const float m1 = s_ml[row], mm = fmaxf(m_ref, m1);
          w0 = exp2f(m_ref - mm);                                // key 0 is visible to every row: m_ref is finite
          w1 = m1 == -INFINITY ? 0.f : exp2f(m1 - mm);
          l = l * w0 + s_ml[128 + row] * w1;
        }
        const float inv = l > 0.f ? 1.f / l : 0.f;
        w0 *= inv;
        w1 *= inv;
        bf16* dst = p.out + (long long)(q_begin + qrow) * p.ld_out + h * p.V;
        const bf16* gate = p.gate + (long long)(q_begin + qrow) * p.ld_gate + h * p.V;
#pragma unroll 1
        for (int c = 0; c < NV * 2; ++c) {
          uint32_t r[32];
          tmem_ld_32x32(to + uint32_t(c * 32), r);
          tmem_ld_wait();
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int col = c * 32 + q * 8;
            if (qrow >= q_len || col >= p.V) continue;           // V is a multiple of 8
            const uint4 gu = *reinterpret_cast<const uint4*>(gate + col);
            const uint32_t gw[4] = {gu.x, gu.y, gu.z, gu.w};
            uint32_t ow[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float a = __uint_as_float(r[q * 8 + 2 * e]) * w0, b = __uint_as_float(r[q * 8 + 2 * e + 1]) * w0;
              if (two) {
                a = fmaf(s_o[(col + 2 * e) * 128 + row], w1, a);
                b = fmaf(s_o[(col + 2 * e + 1) * 128 + row], w1, b);
              }
              const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[e]));
              ow[e] = pack_bf16(a * sigmoid_t<bf16>(g.x), b * sigmoid_t<bf16>(g.y));
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
  return p.D % 8 == 0 && p.D <= 128 && p.R % 8 == 0 && p.R <= 64 && p.V % 8 == 0 && p.V <= 128 && p.rank % 8 == 0 &&
         p.D > 0 && p.R > 0 && p.V > 0;
}

template <int ND, int NV>
static void launch_lp(const LpMaps& tm, const LpParams& q, const LatentPrefill& p, cudaStream_t s) {
  constexpr int smem = 3 * (ND + 1) * LP_SUB + 2 * NV * LP_SUB + 128 + 1024 + 1024;
  auto kern = latent_prefill_kernel<ND, NV>;
  cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  kern<<<dim3((p.max_q + LP_BM - 1) / LP_BM, p.H, p.B), LP_THREADS, smem, s>>>(tm, q);
}

void launch_latent_prefill(const LatentPrefill& p, cudaStream_t s) {
  if (p.T == 0 || p.B == 0 || p.max_q == 0) return;
  LpMaps tm;
  const uint64_t Q = uint64_t(p.D + p.R);
  const bf16* q = reinterpret_cast<const bf16*>(p.q);
  tm.qn = make_tmap_bf16_3d(q, p.D, p.H, p.T, Q, p.ld_q, 64, 1, LP_BM);
  tm.qr = make_tmap_bf16_3d(q + p.D, p.R, p.H, p.T, Q, p.ld_q, 64, 1, LP_BM);
  tm.kn = make_tmap_bf16_3d(p.k, p.D, p.H, p.total_kv, p.D, p.ld_kv, 64, 1, LP_BN);
  tm.v = make_tmap_bf16_3d(p.v, p.V, p.H, p.total_kv, p.V, p.ld_kv, 64, 1, LP_BN);
  tm.kr = make_tmap_bf16_2d(p.rot, p.total_kv, p.R, p.ld_rot, LP_BN, 64);
  LpParams a;
  a.cu_q = p.cu_q;
  a.cu_kv = p.cu_kv;
  a.gate = reinterpret_cast<const bf16*>(p.gate);
  a.out = reinterpret_cast<bf16*>(p.out);
  a.ld_gate = p.ld_gate;
  a.ld_out = p.ld_out;
  a.D = p.D;
  a.R = p.R;
  a.V = p.V;
  a.scale_log2 = p.scale * 1.4426950408889634f;
  a.status = p.status;
  if (p.D <= 64 && p.V <= 64) launch_lp<1, 1>(tm, a, p, s);
  else if (p.D <= 64) launch_lp<1, 2>(tm, a, p, s);
  else if (p.V <= 64) launch_lp<2, 1>(tm, a, p, s);
  else launch_lp<2, 2>(tm, a, p, s);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("latent prefill: ") + cudaGetErrorString(e));
}

}  // namespace fc
