// Attention of decode-size batches over cache rows that all heads share, on tcgen05 (the general tensor-core form is in
// latent_decode.cu): latent rows, whose first columns are the values too, or rows with the keys of several key heads side by
// side and the values behind them.
//
// Grid (query row, group of 32 heads, split of the context).  A CTA walks its rows of the cache in tiles of 128 rows, or of 64
// where wider tiles would leave no room for the next one's keys.  The wide operand of both products is the cache, not the few
// heads:
//     S^T [rows x 32 heads]        = rows (key columns) * Q^T                  A: row tile, K-major; B: Q, K-major
//     O^T [128 columns x 32 heads] += rows^T * P^T, one block per 128 value columns  A: MN-major; B: P, K-major
// (S^T is issued with 128 rows; of a tile of 64 the upper ones read the shared memory behind it, their lanes are ignored.)  Shared
// memory holds a tile as pairs of 64-column sub-tiles in a ring, and the columns behind latent pairs in a ring of two
// sub-tiles.  Latent pairs serve both products and are refilled as soon as their block of O^T is done; other rows have pairs
// of keys, then pairs of values.  Where value heads differ, every head takes its own columns of O^T at the end.
//   warp 0     TMA, boxes that never straddle a page
//   warp 1     tcgen05.mma issuer; the scores of the next tile go first, so that they overlap the softmax of this one (where
//              the ring holds the values of one tile and the keys of the next)
//   warps 2-5  one cache row per thread: P = 2^(s - ref) for all heads against a reference per head (the score of the first
//              visible row; should a score outgrow it by 2^64, all accumulators move to the new maximum), P to shared memory
//              as bf16, sums per thread; at the end one value column per thread
#include <algorithm>
#include <stdexcept>
#include <string>

#include "gemm.h"
#include "hybrid.cuh"
#include "launch.h"
#include "one_lane.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int LT_HEADS = 32, LT_MAX_RING = 12, LT_THREADS = 192;
constexpr int LT_QSUB = LT_HEADS * 128;           // of a [32 heads x 64 columns] sub-tile
// tensor memory: S^T of even / odd tiles [0, 32) [32, 64), O^T blocks [64 + 32 b, ...)
constexpr float LT_RANGE = 64.f;                  // log2 units above the reference that P may reach
constexpr int LT_MAX_BLOCKS = 14;
constexpr float LT_LOG2E = 1.4426950408889634f;

// A tile in the ring: `pairs` slots of 128 columns, of which the first `keys` enter the scores and the last `values` make the
// blocks of O^T; `extra`: 64 more key columns; `shared`: keys and values are the same pairs
struct LtTile {
  int rows, pairs, keys, values, extra, ring, ahead, tmem;
  bool shared;
};

__device__ __forceinline__ uint64_t lt_sdesc(uint32_t addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  uint64_t d = 0;
  d |= uint64_t((addr & 0x3FFFF) >> 4);
  d |= uint64_t((lbo_bytes >> 4) & 0x3FFF) << 16;
  d |= uint64_t((sbo_bytes >> 4) & 0x3FFF) << 32;
  d |= uint64_t(1) << 46;
  d |= uint64_t(2) << 61;
  return d;
}

template <int LT_ROWS>
__global__ void __launch_bounds__(LT_THREADS, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tm, const RowAttn p, const LtTile w, int box_rows,
                        float scale_log2) {
  constexpr int LT_SUB = LT_ROWS * 128;                            // bytes of a [rows x 64 columns] sub-tile
  constexpr int PSUBS = LT_ROWS / 64;                              // sub-tiles of P
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int subs = w.keys * 2 + w.extra;                           // sub-tiles of Q
  uint8_t* s_kv = smem;                                            // [ring] pairs of sub-tiles
  uint8_t* s_x = s_kv + w.ring * 2 * LT_SUB;                       // the columns behind the pairs
  uint8_t* s_q = s_x + (w.extra ? 2 * LT_SUB : 0);                 // [subs] sub-tiles
  uint8_t* s_p = s_q + subs * LT_QSUB;
  float* s_ref = reinterpret_cast<float*>(s_p + 2 * PSUBS * LT_QSUB);      // (P of even / odd tiles)  [32] reference
  float* s_red = s_ref + LT_HEADS;                                 // [4][32]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_red + 4 * LT_HEADS);
  uint64_t *full = bars, *empty = bars + LT_MAX_RING, *x_full = bars + 2 * LT_MAX_RING, *x_empty = x_full + 2;
  // o_done: O^T complete up to a tile.  p_ready of even / odd tiles apart: the scores of the next tile are issued before the issuer
  // waits for this one's P, so one barrier could be two phases ahead of its wait
  uint64_t *s_full = x_full + 4, *p_ready = x_full + 6, *o_done = x_full + 8, *q_ready = x_full + 9;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(x_full + 10);
  volatile int* s_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_at = reinterpret_cast<int*>(tmem_slot + 2);               // [LT_ROWS / 8]

  const int t = blockIdx.x, h0 = blockIdx.y * LT_HEADS, split = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_launch_dependents();
  if (tid == 0) {
    for (int i = 0; i < w.ring; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&x_full[i], 1);
      mbar_init(&x_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&p_ready[i], 128);
    }
    mbar_init(q_ready, 128);
    mbar_init(o_done, 1);
    *s_abort = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tm);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, uint32_t(w.tmem));
    tmem_relinquish();
  }
  pdl_wait();
  asm volatile("fence.proxy.async.global;" ::: "memory");          // rows were written with ordinary stores
  const int ctx = min(p.row_ctx[t], p.max_blocks * p.block_size);
  const int b = p.row_seq != nullptr ? p.row_seq[t] : t;
  const int first = p.window > 0 ? max(0, ctx - p.window) : 0;     // first visible row
  const int tiles = (ctx + LT_ROWS - 1) / LT_ROWS, start = first / LT_ROWS;
  const int per = (tiles - start + p.splits - 1) / p.splits;
  const int tile0 = start + split * per, n_tiles = max(0, min(tiles, tile0 + per) - tile0);
  const int* bt = p.block_tables + (long long)b * p.max_blocks;

  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA loader
    const uint32_t el = elect_one() ? 1u : 0u;
    {
      int slot = 0;
      bool ok = true;
      uint32_t phase = 1;
      constexpr int MAX_PIECES = LT_ROWS / 8;
      const int pieces = LT_ROWS / box_rows;
      int next[MAX_PIECES];                                        // pool row of every piece of a tile, one tile ahead
      auto find = [&](int j) {
        const int row0 = (tile0 + j) * LT_ROWS;
#pragma unroll
        for (int pc = 0; pc < MAX_PIECES; ++pc) {
          if (j >= n_tiles || pc * box_rows >= LT_ROWS) continue;
          // a box past the context is loaded from the last one inside: what its rows hold must only be finite
          const int tok = min(row0 + pc * box_rows, (ctx - 1) / box_rows * box_rows);
          int blk = bt[tok / p.block_size];
          if (blk < 0 || blk >= p.num_blocks) {
            if (lane == 0) report(p.status, ST_BAD_INDEX);
            blk = 0;
          }
          next[pc] = blk * p.block_size + tok % p.block_size;
        }
      };
      find(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        // through shared memory: the issue loop stays one instruction sequence for any number of pieces
        ok = !__any_sync(0xffffffffu, *s_abort != 0);                // also: every lane is done with the tile before
#pragma unroll
        for (int pc = 0; pc < MAX_PIECES; ++pc)
          if (lane == 0) s_at[pc] = next[pc];
        __syncwarp();
        find(j + 1);
        auto load = [&](uint8_t* dst, uint64_t* bar, int col) {
#pragma unroll 1
          for (int pc = 0; pc < pieces; ++pc)
            one_load_2d(dst + pc * box_rows * 128, &tm, bar, col, reinterpret_cast<volatile int*>(s_at)[pc], el);
        };
        for (int i = 0; i < w.pairs; ++i) {
          const int col = w.shared || i < w.keys ? i * 128 : p.v_col + (i - w.keys) * 128;
          if (!__all_sync(0xffffffffu, mbar_wait(&empty[slot], phase, p.status, ST_TIMEOUT_EMPTY))) {
            if (lane == 0) *s_abort = 1;
            ok = false;
            break;
          }
          one_expect(&full[slot], 2 * LT_SUB, el);
          load(s_kv + slot * 2 * LT_SUB, &full[slot], col);
          load(s_kv + slot * 2 * LT_SUB + LT_SUB, &full[slot], col + 64);
          if (++slot == w.ring) {
            slot = 0;
            phase ^= 1;
          }
        }
        if (w.extra && ok) {
          const int x = j & 1;
          if (!__all_sync(0xffffffffu, mbar_wait(&x_empty[x], (uint32_t(j >> 1) & 1u) ^ 1u, p.status, ST_TIMEOUT_EMPTY))) {
            if (lane == 0) *s_abort = 1;
            ok = false;
            break;
          }
          one_expect(&x_full[x], LT_SUB, el);
          load(s_x + x * LT_SUB, &x_full[x], w.keys * 128);
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    const uint32_t el = elect_one() ? 1u : 0u;
    {
      constexpr uint32_t idesc_s = make_idesc_bf16(128, LT_HEADS, false, false);
      constexpr uint32_t idesc_o = make_idesc_bf16(128, LT_HEADS, true, false);      // A (rows^T) is MN-major
      const int ksteps = (p.K + 15) / 16;
      auto wait = [](uint64_t* bar, uint32_t parity, uint32_t* status, uint32_t code) {
        return __all_sync(0xffffffffu, mbar_wait(bar, parity, status, code)) != 0;
      };
      int slot = 0, sl = 0;                                        // next pair of O^T and of S^T, their phases
      uint32_t pho = 0, ph = 0;
      auto skip = [&](int& at, uint32_t& phase, int n) {
        at += n;
        while (at >= w.ring) {
          at -= w.ring;
          phase ^= 1;
        }
      };
      skip(slot, pho, w.pairs - w.values);
      // descriptors by addition on their address field (16-byte units)
      const uint64_t d_rows = lt_sdesc(smem_u32(s_kv), 16, 1024), d_x = lt_sdesc(smem_u32(s_x), 16, 1024);
      const uint64_t d_cols = lt_sdesc(smem_u32(s_kv), LT_SUB, 1024);
      const uint64_t d_q = lt_sdesc(smem_u32(s_q), 16, 1024), d_p = lt_sdesc(smem_u32(s_p), 16, 1024);
      auto scores = [&](uint32_t tm_s, uint64_t da, int sub) {
        const uint64_t dq = d_q + uint64_t(sub * (LT_QSUB >> 4));
        const int left = ksteps - sub * 4;
        if (elect_one())
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            if (kk < left) tc_mma_f16(tm_s, da + uint64_t(kk * 2), dq + uint64_t(kk * 2), idesc_s, (sub > 0 || kk > 0) ? 1u : 0u);
        __syncwarp();
      };
      auto issue_s = [&](int j) {
        const int x = j & 1;
        for (int i = 0; i < w.keys; ++i) {
          if (!wait(&full[sl], ph, p.status, ST_TIMEOUT_FULL)) return false;
          tc_fence_after();
          const uint64_t da = d_rows + uint64_t(sl * (2 * LT_SUB >> 4));
          scores(tmem + LT_HEADS * uint32_t(x), da, i * 2);
          scores(tmem + LT_HEADS * uint32_t(x), da + uint64_t(LT_SUB >> 4), i * 2 + 1);
          if (!w.shared) one_commit(&empty[sl], el);
          skip(sl, ph, 1);
        }
        skip(sl, ph, w.pairs - w.keys);
        if (w.extra) {
          if (!wait(&x_full[x], uint32_t(j >> 1) & 1u, p.status, ST_TIMEOUT_FULL)) return false;
          tc_fence_after();
          scores(tmem + LT_HEADS * uint32_t(x), d_x + uint64_t(x * (LT_SUB >> 4)), w.keys * 2);
        }
        one_commit(&s_full[x], el);
        if (w.extra) one_commit(&x_empty[x], el);
        return true;
      };
      bool ok = n_tiles == 0 || (wait(q_ready, 0, p.status, ST_TIMEOUT_FULL) && issue_s(0));
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (w.ahead && j + 1 < n_tiles) ok = issue_s(j + 1);
        ok = ok && wait(&p_ready[j & 1], uint32_t(j >> 1) & 1u, p.status, ST_TIMEOUT_FULL);
        if (!ok) break;
        tc_fence_after();
        for (int i = 0; i < w.values && ok; ++i) {
          if (!w.shared) {
            ok = wait(&full[slot], pho, p.status, ST_TIMEOUT_FULL);
            if (!ok) break;
            tc_fence_after();
          }
          const uint64_t dv = d_cols + uint64_t(slot * (2 * LT_SUB >> 4)), dp = d_p + uint64_t((j & 1) * (PSUBS * LT_QSUB >> 4));
          const uint32_t tm_o = tmem + LT_HEADS * uint32_t(2 + i);
          if (elect_one())
#pragma unroll
            for (int kk = 0; kk < LT_ROWS / 16; ++kk)
              tc_mma_f16(tm_o, dv + uint64_t(kk * 128), dp + uint64_t((kk >> 2) * (LT_QSUB >> 4) + (kk & 3) * 2), idesc_o, (j > 0 || kk > 0) ? 1u : 0u);
          __syncwarp();
          one_commit(&empty[slot], el);
          skip(slot, pho, 1);
        }
        skip(slot, pho, w.pairs - w.values);
        if (!ok) break;
        one_commit(o_done, el);
        if (!w.ahead && j + 1 < n_tiles) ok = issue_s(j + 1);
      }
      if (!ok && lane == 0) *s_abort = 1;
    }
  } else {
    // ------------------------------------------------------------------ Q; softmax; epilogue
    if (n_tiles > 0) {                                             // zero-padded to whole sub-tiles and head rows
      const uint4* q = reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p.q) + ((long long)t * p.H + h0) * p.K);
      constexpr int N = LT_HEADS / 4;
      for (int ch = lane; ch < subs * 8; ch += 32) {
        uint4 v[N];
#pragma unroll
        for (int i = 0; i < N; ++i) {
          const int r = warp - 2 + i * 4;
          v[i] = h0 + r < p.H && ch * 8 < p.K ? __ldcg(q + (long long)r * (p.K / 8) + ch) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int i = 0; i < N; ++i) {
          const int r = warp - 2 + i * 4;
          *reinterpret_cast<uint4*>(s_q + (ch >> 3) * LT_QSUB + r * 128 + (((ch & 7) ^ (r & 7)) << 4)) = v[i];
        }
      }
      fence_proxy_async();
      mbar_arrive(q_ready);
    }
    const int group = warp & 3;                                    // TMEM lanes this warp may touch
    const int row = group * 32 + lane;
    const uint32_t lanes = uint32_t(group * 32) << 16;
    auto sync_or = [](bool x) {                                    // over the four warps
      uint32_t r;
      asm volatile(
          "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbar.red.or.pred q, 1, 128, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
          : "=r"(r)
          : "r"(x ? 1u : 0u)
          : "memory");
      return r != 0;
    };
    float l[LT_HEADS];
#pragma unroll
    for (int h = 0; h < LT_HEADS; ++h) l[h] = 0.f;
    uint8_t* prow = s_p + (PSUBS > 1 ? (row >> 6) * LT_QSUB : 0) + (row & 7) * 2;
    const int chunk = (row & 63) >> 3;
    const bool mine = row < LT_ROWS;                               // warp-uniform: of 64 rows the upper lanes hold none
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      if (ok) ok = !*s_abort && mbar_wait(&s_full[j & 1], uint32_t(j >> 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL);
      if (sync_or(!ok)) {                                          // all four warps leave together
        ok = false;
        break;
      }
      tc_fence_after();
      uint32_t s[LT_HEADS];
      tmem_ld_32x32(tmem + lanes + LT_HEADS * uint32_t(j & 1), s);
      tmem_ld_wait();
      const int at = (tile0 + j) * LT_ROWS + row;
      const bool valid = mine && at < ctx && at >= first;
      if (j == 0) {
        if (row == max(0, first - tile0 * LT_ROWS))
#pragma unroll
          for (int h = 0; h < LT_HEADS; ++h) s_ref[h] = __uint_as_float(s[h]) * scale_log2;
        sync_or(false);
      }
      float v[LT_HEADS], top = -INFINITY;
#pragma unroll
      for (int h = 0; h < LT_HEADS; h += 4) {
        const float4 r = *reinterpret_cast<const float4*>(s_ref + h);
        const float rr[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          v[h + e] = fmaf(__uint_as_float(s[h + e]), scale_log2, -rr[e]);      // relative to the reference
          top = fmaxf(top, v[h + e]);
        }
      }
      const bool far = top > LT_RANGE;
      if (sync_or(far && valid)) {
        // a score outgrew its reference: maximum over the tile, then sums and O^T (complete up to the tile before) move
        // to the new reference
#pragma unroll
        for (int h = 0; h < LT_HEADS; ++h) {
          const float m = warp_max(valid ? v[h] + s_ref[h] : -INFINITY);
          if (lane == h) s_red[group * LT_HEADS + h] = m;
        }
        sync_or(false);
        float f[LT_HEADS];
#pragma unroll
        for (int h = 0; h < LT_HEADS; ++h) {
          const float m = fmaxf(fmaxf(s_red[h], s_red[LT_HEADS + h]), fmaxf(s_red[2 * LT_HEADS + h], s_red[3 * LT_HEADS + h]));
          f[h] = exp2f(fminf(s_ref[h] - m, 0.f));
          l[h] *= f[h];
          v[h] += fminf(s_ref[h] - m, 0.f);
        }
        if (j > 0 && ok) ok = mbar_wait(o_done, uint32_t(j - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL);
        tc_fence_after();
        if (j > 0)
          for (int i = 0; i < w.values; ++i) {
            uint32_t r[32];
            tmem_ld_32x32(tmem + lanes + LT_HEADS * uint32_t(2 + i), r);
            tmem_ld_wait();
#pragma unroll
            for (int h = 0; h < LT_HEADS; ++h) r[h] = __float_as_uint(__uint_as_float(r[h]) * f[h]);
            tmem_st_32x32(tmem + lanes + LT_HEADS * uint32_t(2 + i), r);
            tmem_st_wait();
          }
        sync_or(false);
        if (row < LT_HEADS) {
          const int h = row;
          s_ref[h] = fmaxf(s_ref[h], fmaxf(fmaxf(s_red[h], s_red[LT_HEADS + h]),
                                           fmaxf(s_red[2 * LT_HEADS + h], s_red[3 * LT_HEADS + h])));
        }
        sync_or(false);
      }
      if (mine) {
#pragma unroll
        for (int h = 0; h < LT_HEADS; ++h) {
          float e;
          asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(valid ? v[h] : -INFINITY));
          l[h] += e;
          *reinterpret_cast<bf16*>(prow + (j & 1) * PSUBS * LT_QSUB + h * 128 + ((chunk ^ (h & 7)) << 4)) = __float2bfloat16(e);
        }
      }
      // the last two phases of o_done one by one, a parity cannot tell a phase from the one two before it: the scores of the
      // last tile only say that the third-last product is done, and the last one cannot be before this arrival
      if (j == n_tiles - 1 && j > 0 && ok) ok = mbar_wait(o_done, uint32_t(j - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL);
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(&p_ready[j & 1]);
    }
    if (ok && n_tiles > 0) ok = mbar_wait(o_done, uint32_t(n_tiles - 1) & 1u, p.status, ST_TIMEOUT_ACC_FULL);
    if (!ok) *s_abort = 1;
    tc_fence_after();
    // every product is done: the ring is free.  Sums over the rows, then O^T block by block, a lane per value column
    const bool good = !sync_or(!ok) && n_tiles > 0;
    float* s_l = reinterpret_cast<float*>(s_kv);                   // [LT_ROWS][33]
    const int et = tid - 64;                                       // 0..127
    if (mine)
#pragma unroll
      for (int h = 0; h < LT_HEADS; ++h) s_l[row * 33 + h] = l[h];
    sync_or(false);
    {
      float x = 0.f;
      for (int r = et >> 5; r < LT_ROWS; r += 4) x += s_l[r * 33 + (et & 31)];
      s_red[et] = x;
    }
    sync_or(false);
    if (et < LT_HEADS) {
      const float x = s_red[et] + s_red[LT_HEADS + et] + s_red[2 * LT_HEADS + et] + s_red[3 * LT_HEADS + et];
      const bool has = good && x > 0.f;
      const int head = h0 + et;
      if (p.splits > 1 && head < p.H)
        p.part_lse[((long long)t * p.H + head) * p.splits + split] = has ? s_ref[et] + log2f(x) : -INFINITY;
      float f = 0.f;
      if (has) {
        f = 1.f / x;
        if (p.splits == 1 && head < p.H) {
          if (p.sink != nullptr) f = 1.f / (x + exp2f(p.sink[head] * LT_LOG2E - s_ref[et]));
          if (p.head_gate != nullptr) f *= p.head_gate[(long long)t * p.H + head];
        }
      }
      s_red[et] = f;
    }
    sync_or(false);
    const int heads_per = p.H / p.v_heads, here = min(LT_HEADS, p.H - h0);
    const long long head0 = (long long)t * p.H + h0;
    // short loops: this code runs once per CTA, and fetching it is what it waits for
#pragma unroll 1
    for (int i = 0; i < w.values; ++i) {
      const int c = i * 128 + row, vh = c / p.V, cv = c - vh * p.V;    // the value head of this column takes it
      const int lo = vh * heads_per - h0, hi = vh < p.v_heads ? min(here, lo + heads_per) : 0;
      bf16* out = reinterpret_cast<bf16*>(p.out) + t * p.ld_out + (long long)h0 * p.V + cv;
      float* part = p.part_o + (head0 * p.splits + split) * p.V + cv;
      const int step = p.splits == 1 ? p.V : p.splits * p.V;
#pragma unroll 1
      for (int h8 = 0; h8 < here; h8 += 8) {
        uint32_t r[8];
        __syncwarp();
        tmem_ld_32x8(tmem + lanes + LT_HEADS * uint32_t(2 + i) + uint32_t(h8), r);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int h = h8 + e;
          if (h < lo || h >= hi) continue;
          const float f = s_red[h], x = f != 0.f ? __uint_as_float(r[e]) * f : 0.f;      // 0: no row was seen
          if (p.splits == 1) out[(long long)h * step] = __float2bfloat16(x);
          else part[(long long)h * step] = x;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, uint32_t(w.tmem));
  }
}

static int lt_box_rows(int block_size, int rows) {
  int box = rows;
  while (box > block_size || block_size % box != 0) box >>= 1;
  return box;
}

static int lt_smem(const LtTile& w) {
  const int sub = w.rows * 128;
  return w.ring * 2 * sub + (w.extra ? 2 * sub : 0) + (w.keys * 2 + w.extra + 2 * (w.rows / 64)) * LT_QSUB + 5 * LT_HEADS * 4 +
         (2 * LT_MAX_RING + 10) * 8 + 16 + w.rows / 2 + 1024;
}
// how a tile lies in the ring; ring 0: these sizes do not fit
static LtTile lt_tile(const RowAttn& p) {
  LtTile w{};
  const int vw = p.v_heads * p.V;
  w.rows = 64;
  w.shared = p.v_col == 0;
  w.values = (vw + 127) / 128;
  if (w.shared) {
    w.pairs = w.keys = w.values;
    w.extra = p.K > w.keys * 128 ? 1 : 0;
    if (p.K - w.keys * 128 > 64 || vw > p.K) return w;
  } else {
    w.keys = (p.K + 127) / 128;
    w.pairs = w.keys + w.values;
  }
  if (w.values > LT_MAX_BLOCKS) return w;
  w.tmem = w.values <= 6 ? 256 : 512;
  auto fit = [](LtTile& x, int most) {
    x.ring = most;
    while (x.ring > 0 && lt_smem(x) > 227 * 1024) --x.ring;
  };
  if (!w.shared) {
    LtTile wide = w;
    wide.rows = 128;
    wide.ahead = 1;
    fit(wide, LT_MAX_RING / 2);
    if (wide.ring >= w.keys + w.values) return wide;
  }
  fit(w, w.shared ? 10 : LT_MAX_RING);
  if (w.ring < 4 || (w.shared && w.ring < 2 * w.pairs)) w.ring = 0;
  w.ahead = w.shared || w.keys + w.values <= w.ring ? 1 : 0;
  return w;
}

bool latent_decode_tc_supported(const RowAttn& p) {
  return p.V % 8 == 0 && p.K % 8 == 0 && p.v_col % 8 == 0 && p.row_width % 8 == 0 && p.ld_out % 4 == 0 && p.H % p.v_heads == 0 &&
         lt_box_rows(p.block_size, 64) >= 8 && lt_tile(p).ring > 0;
}

int latent_decode_tc_splits(const RowAttn& p, int max_ctx, int num_sms) {
  const int ctas = p.T * ((p.H + LT_HEADS - 1) / LT_HEADS);
  if (ctas * 3 > num_sms * 2) return 1;                            // nearly a full wave already
  return std::max(1, std::min({num_sms / std::max(1, ctas), max_ctx / 128, 32}));
}

void launch_latent_decode_tc(const RowAttn& p, cudaStream_t s) {
  if (p.T == 0) return;
  const LtTile w = lt_tile(p);
  const int box = lt_box_rows(p.block_size, w.rows), smem = lt_smem(w);
  if (w.ring == 0) throw std::runtime_error("attention over shared rows (tcgen05): unsupported sizes");
  const CUtensorMap tm = make_tmap_bf16_2d(p.pool, (uint64_t)p.num_blocks * p.block_size, p.row_width, p.row_width, box, 64);
  auto go = [&](auto kern) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    launch_pdl(PDL_DECODE_ATTN, kern, dim3(p.T, (p.H + LT_HEADS - 1) / LT_HEADS, p.splits), dim3(LT_THREADS), smem, s, tm, p, w, box,
               p.scale * LT_LOG2E);
  };
  if (w.rows == 128) go(latent_decode_tc_kernel<128>);
  else go(latent_decode_tc_kernel<64>);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("attention over shared rows (tcgen05): ") + cudaGetErrorString(e));
}

}  // namespace fc
