// Expert projections of decode-size batches: y[r, n] = sum_k x[r, k] W[e(r)][n, k], rows sorted by expert.
//
// Bound by reading the weights of the experts in use once, so (as in gemm_skinny.cu) the weights are the 128-row tcgen05
// operand and an expert's rows of x the N operand: grid (128-row tile of W, K split, expert), an expert without rows
// returns at once.  TMA boxes of x start at the expert's first row; what they read past its last one is not written.
//   warp 0    TMA producer (W tile 128 x 64 and x tile BN x 64 per stage, 128-byte swizzle)
//   warp 1    tcgen05.mma issuer, accumulator in tensor memory (BN fp32 columns)
//   warps 2-5 tcgen05.ld, fp32 partial sums [split, rows, N] for the reader
// Two CTAs fit an SM up to BN = 128.
#include <cuda.h>

#include <algorithm>
#include <stdexcept>
#include <string>

#include "gemm.h"
#include "launch.h"
#include "ptx.cuh"

namespace fc {

constexpr int MG_ROWS = 128, MG_BK = 64, MG_WARPS = 6;

struct MoeSkinnyParams {
  int N, K, pairs, kb_per_split;
  const int* plan;                 // [E + 1] first row of every expert
  float* partial;
  uint32_t* status;
};

template <int BN, int STAGES>
struct MoeSmem {
  static constexpr int A_BYTES = MG_ROWS * MG_BK * 2, B_BYTES = BN * MG_BK * 2, STAGE_BYTES = A_BYTES + B_BYTES;
  static constexpr int BAR_OFF = STAGES * STAGE_BYTES, TOTAL = BAR_OFF + 256 + 1024;
};

template <int BN, int STAGES>
__global__ void __launch_bounds__(MG_WARPS * 32)
moe_skinny_kernel(const __grid_constant__ CUtensorMap tma_w, const __grid_constant__ CUtensorMap tma_x,
                  const MoeSkinnyParams p) {
  using L = MoeSmem<BN, STAGES>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + L::BAR_OFF);
  uint64_t* empty_bar = full_bar + STAGES;
  uint64_t* acc_full = empty_bar + STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_full + 1);
  volatile int* s_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);
  pdl_launch_dependents();
  pdl_wait();
  const int tile = blockIdx.x, split = blockIdx.y, e = blockIdx.z;
  const int row0 = __ldcg(p.plan + e), rows = __ldcg(p.plan + e + 1) - row0;
  if (rows <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int num_kb = (p.K + MG_BK - 1) / MG_BK;
  const int kb0 = split * p.kb_per_split, kb1 = min(num_kb, kb0 + p.kb_per_split);
  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    mbar_init(acc_full, 1);
    *s_abort = 0;
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, BN);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      asm volatile("fence.proxy.async.global;" ::: "memory");       // x: ordinary stores before, TMA reads now
      int stage = 0, issued = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int kb = kb0; kb < kb1; ++kb) {
        if (*s_abort || !mbar_wait(&empty_bar[stage], phase ^ 1, p.status, ST_TIMEOUT_EMPTY)) {
          *s_abort = 1;
          ok = false;
          break;
        }
        uint8_t* sa = smem + stage * L::STAGE_BYTES;
        mbar_expect_tx(&full_bar[stage], L::STAGE_BYTES);
        tma_load_2d(sa, &tma_w, &full_bar[stage], kb * MG_BK, e * p.N + tile * MG_ROWS);
        tma_load_2d(sa + L::A_BYTES, &tma_x, &full_bar[stage], kb * MG_BK, row0);
        ++issued;
        if (++stage == STAGES) {
          stage = 0;
          phase ^= 1;
        }
      }
      if (!ok) {                       // let every copy that was issued land before the CTA may exit
        int s = stage;
        uint32_t ph = phase;
        for (int n = 0; n < min(issued, STAGES); ++n) {
          if (--s < 0) {
            s = STAGES - 1;
            ph ^= 1;
          }
          mbar_wait(&full_bar[s], ph, nullptr, 0);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc_bf16(128, BN);
      int stage = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int kb = kb0; kb < kb1; ++kb) {
        if (*s_abort || !mbar_wait(&full_bar[stage], phase, p.status, ST_TIMEOUT_FULL)) {
          *s_abort = 1;
          ok = false;
          break;
        }
        tc_fence_after();
        const uint32_t sa = smem_u32(smem + stage * L::STAGE_BYTES);
        const uint64_t da = make_sdesc_sw128(sa), db = make_sdesc_sw128(sa + L::A_BYTES);
#pragma unroll
        for (int k = 0; k < MG_BK / 16; ++k)
          tc_mma_f16(tmem_base, da + uint64_t(2 * k), db + uint64_t(2 * k), idesc, (kb > kb0 || k > 0) ? 1u : 0u);
        tc_commit(&empty_bar[stage]);
        if (++stage == STAGES) {
          stage = 0;
          phase ^= 1;
        }
      }
      if (ok) tc_commit(acc_full);
    }
  } else if (!*s_abort && mbar_wait(acc_full, 0, p.status, ST_TIMEOUT_ACC_FULL)) {
    tc_fence_after();
    const int lane_group = warp & 3, n = tile * MG_ROWS + lane_group * 32 + lane;
    const uint32_t t_addr = tmem_base + (uint32_t(lane_group * 32) << 16);
    float* dst = p.partial + ((long long)split * p.pairs + row0) * p.N + n;
#pragma unroll 1
    for (int c = 0; c < BN / 32 && c * 32 < rows; ++c) {
      uint32_t r[32];
      __syncwarp();
      tmem_ld_32x32(t_addr + uint32_t(c * 32), r);
      tmem_ld_wait();
      if (n < p.N) {
#pragma unroll
        for (int t = 0; t < 32; ++t)
          if (c * 32 + t < rows) dst[(long long)(c * 32 + t) * p.N] = __uint_as_float(r[t]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, BN);
  }
}

int moe_skinny_splits(int max_rows, int pairs, int E, int N, int K) {
  const int tiles = (N + MG_ROWS - 1) / MG_ROWS, num_kb = (K + MG_BK - 1) / MG_BK;
  const int ctas = tiles * std::min(E, pairs), slots = (max_rows <= 128 ? 2 : 1) * gemm_num_sms();
  int splits = std::max(1, std::min({slots / std::max(1, ctas), num_kb / 4, 16}));
  const int per = (num_kb + splits - 1) / splits;
  return (num_kb + per - 1) / per;
}

void launch_moe_skinny(const void* x, const void* w, float* partial, int splits, const int* plan, int max_rows, int pairs,
                       int E, int N, int K, uint32_t* status, cudaStream_t s) {
  if (pairs == 0) return;
  if (max_rows > 256) throw std::runtime_error("decode-size expert products are for up to 256 rows per expert");
  MoeSkinnyParams p{};
  p.N = N;
  p.K = K;
  p.pairs = pairs;
  p.kb_per_split = ((K + MG_BK - 1) / MG_BK + splits - 1) / splits;
  p.plan = plan;
  p.partial = partial;
  p.status = status;
  const CUtensorMap tw = make_tmap_bf16_2d(w, (uint64_t)E * N, K, K, MG_ROWS, MG_BK);
  const dim3 grid((N + MG_ROWS - 1) / MG_ROWS, splits, E);
  auto go = [&](auto kern, int bn, int smem) {
    const CUtensorMap tx = make_tmap_bf16_2d(x, pairs, K, K, bn, MG_BK);
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    launch_pdl(PDL_SKINNY_GEMM, kern, grid, dim3(MG_WARPS * 32), smem, s, tw, tx, p);
  };
  if (max_rows <= 32) go(moe_skinny_kernel<32, 5>, 32, MoeSmem<32, 5>::TOTAL);
  else if (max_rows <= 64) go(moe_skinny_kernel<64, 4>, 64, MoeSmem<64, 4>::TOTAL);
  else if (max_rows <= 128) go(moe_skinny_kernel<128, 3>, 128, MoeSmem<128, 3>::TOTAL);
  else go(moe_skinny_kernel<256, 4>, 256, MoeSmem<256, 4>::TOTAL);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("expert products: ") + cudaGetErrorString(e));
}

}  // namespace fc
