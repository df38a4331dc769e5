// Absorbed latent attention of decode-size batches (bf16): every query row attends to the cache rows of its request as
// they are, key = [latent | rotated part], value = latent, shared by all heads.
//
// Rows before the window are skipped tile by tile and masked; the sink and the head gates join at the end.
// Grid (query row, group of 16 * MT heads, split of the context).  One tile of 32 cache rows in shared memory is both the
// keys and the values of all heads of the CTA, so a row is read once.  Two groups of eight warps take alternate tiles, each
// with its own two-stage TMA ring (128-byte swizzle, boxes that never straddle a page), running maximum and accumulators:
// while one group is in a latency-bound phase the other keeps the pipes busy.  Per tile and group:
//   scores   warp w: 16 keys (w & 1) against all heads, a quarter of the columns (w >> 1), mma.sync m16n8k16; the
//            quarters are added when they are read back
//   softmax  16 / MT threads per head, running maximum and sum in registers, P to shared memory as bf16
//   values   warp w owns the latent columns of 16-column groups w, w + 8, ...; P V accumulates in registers
// The groups are merged in shared memory at the end.  With several splits a CTA writes normalised partials with their
// log-sum-exp and a second kernel merges them.
//
// Also here: the per-head products around it (queries into the latent space, outputs out of it).
#include <algorithm>
#include <stdexcept>
#include <string>

#include "gemm.h"
#include "hybrid.cuh"
#include "launch.h"
#include "mma.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int LD_TILE = 32, LD_STAGES = 2, LD_GROUPS = 2;
constexpr int LD_WARPS = 8, LD_GT = LD_WARPS * 32, LD_THREADS = LD_GROUPS * LD_GT;      // warps and threads of a group
constexpr int LD_PARTS = 4;                      // column ranges of the scores
constexpr int LD_SUB = LD_TILE * 128;             // bytes of a [32 rows x 64 columns] sub-tile
constexpr int LD_MAX_SPLITS = 32;

// byte offset of 16-byte chunk `chunk` of row `row` in sub-tiles of `rows` rows x 128 bytes
__device__ __forceinline__ uint32_t ld_swz(int rows, int row, int chunk) {
  return uint32_t((chunk >> 3) * rows * 128 + row * 128 + (((chunk & 7) ^ (row & 7)) << 4));
}

template <int MT, int NPW>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm, const RowAttn p, int box_rows, int nc, float scale_log2) {
  constexpr int HR = MT * 16;                     // head rows of this CTA
  constexpr int TPR = LD_GT / HR;                 // softmax threads per head row
  constexpr int KPT = LD_TILE / TPR;              // keys per softmax thread
  constexpr int SLD = LD_TILE + 4;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int stage_bytes = nc * LD_SUB;
  const int tid = threadIdx.x, grp = tid / LD_GT, gt = tid % LD_GT, warp = gt >> 5, lane = tid & 31;
  uint8_t* s_all = smem;                                                     // [group][stage]
  uint8_t* s_q = s_all + LD_GROUPS * LD_STAGES * stage_bytes;                // [nc][HR][128 B]
  uint8_t* s_p = s_q + nc * HR * 128 + grp * HR * 128;                       // [group][HR][128 B]
  float* s_s = reinterpret_cast<float*>(s_q + nc * HR * 128 + LD_GROUPS * HR * 128) + grp * LD_PARTS * HR * SLD;
  float* s_m = reinterpret_cast<float*>(s_q + nc * HR * 128 + LD_GROUPS * HR * 128) + LD_GROUPS * LD_PARTS * HR * SLD;
  float* s_cor = s_m + 2 * HR + grp * HR;                                    // s_m: [2][HR] maximum and sum of group 1
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_m + (2 + LD_GROUPS) * HR);  // [group][stage]
  uint8_t* s_kv = s_all + grp * LD_STAGES * stage_bytes;
  uint64_t* full = bars + grp * LD_STAGES;
  auto group_sync = [&]() { asm volatile("bar.sync %0, %1;" ::"r"(grp + 1), "r"(LD_GT) : "memory"); };

  const int t = blockIdx.x, h0 = blockIdx.y * HR, split = blockIdx.z;
  pdl_launch_dependents();
  if (tid == 0) {
    for (int s = 0; s < LD_GROUPS * LD_STAGES; ++s) mbar_init(&bars[s], 1);
    fence_barrier_init();
    tma_prefetch_desc(&tm);
  }
  pdl_wait();
  asm volatile("fence.proxy.async.global;" ::: "memory");          // rows were written with ordinary stores
  const int ctx = min(p.row_ctx[t], p.max_blocks * p.block_size);
  const int b = p.row_seq != nullptr ? p.row_seq[t] : t;
  const int first = p.window > 0 ? max(0, ctx - p.window) : 0;     // first visible row
  const int tiles = (ctx + LD_TILE - 1) / LD_TILE, start = first / LD_TILE;
  const int per = (tiles - start + p.splits - 1) / p.splits;
  const int tile0 = start + split * per, n_tiles = max(0, min(tiles, tile0 + per) - tile0);
  const int n_mine = (n_tiles - grp + LD_GROUPS - 1) / LD_GROUPS;  // tiles grp, grp + 2, ...
  const int* bt = p.block_tables + (long long)b * p.max_blocks;
  const int w = p.K;

  // Q, zero-padded to whole sub-tiles and head rows
  for (int i = tid; i < HR * nc * 8; i += LD_THREADS) {
    const int r = i / (nc * 8), ch = i - r * (nc * 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (h0 + r < p.H && ch * 8 < w)
      v = __ldcg(reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p.q) +
                                                ((long long)t * p.H + h0 + r) * w + ch * 8));
    *reinterpret_cast<uint4*>(s_q + ld_swz(HR, r, ch)) = v;
  }
  if (n_tiles <= LD_GROUPS * LD_STAGES) {
    // boxes past the context are never loaded: what they would hold must be finite
    for (int i = tid; i < LD_GROUPS * LD_STAGES * stage_bytes / 16; i += LD_THREADS)
      reinterpret_cast<uint4*>(s_all)[i] = make_uint4(0, 0, 0, 0);
    fence_proxy_async();
  }
  __syncthreads();

  auto load_tile = [&](int it) {                                   // the group's it-th tile
    const int stage = it % LD_STAGES, row0 = (tile0 + grp + it * LD_GROUPS) * LD_TILE;
    const int pieces = min(LD_TILE / box_rows, (ctx - row0 + box_rows - 1) / box_rows);
    mbar_expect_tx(&full[stage], uint32_t(pieces) * nc * box_rows * 128);
    for (int pc = 0; pc < pieces; ++pc) {
      const int tok = row0 + pc * box_rows;
      int blk = bt[tok / p.block_size];
      if (blk < 0 || blk >= p.num_blocks) {
        report(p.status, ST_BAD_INDEX);
        blk = 0;
      }
      const int grow = blk * p.block_size + tok % p.block_size;
      for (int c = 0; c < nc; ++c)
        tma_load_2d(s_kv + stage * stage_bytes + c * LD_SUB + pc * box_rows * 128, &tm, &full[stage], c * 64, grow);
    }
  };
  if (gt == 0)
    for (int s = 0; s < LD_STAGES; ++s)
      if (s < n_mine) load_tile(s);

  const int g = lane >> 2, q4 = lane & 3, mat = lane >> 3;
  float o[MT][NPW][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NPW; ++n)
#pragma unroll
      for (int e = 0; e < 8; ++e) o[m][n][e >> 2][e & 3] = 0.f;
  const int srow = gt / TPR, sk0 = (gt % TPR) * KPT;               // softmax: head row and first key of this thread
  float m_run = -INFINITY, l_run = 0.f;
  const int ksteps = (p.row_width + 15) / 16, kpart = (ksteps + LD_PARTS - 1) / LD_PARTS;
  const int kg = (warp & 1) * 16, part = warp >> 1;
  const int k_lo = part * kpart, k_hi = min(ksteps, k_lo + kpart);
  const uint32_t q_base = smem_u32(s_q), p_base = smem_u32(s_p);
  bool alive = true;                                               // false: a tile never landed (the status word says so)
  for (int it = 0; it < n_mine; ++it) {
    const int stage = it % LD_STAGES;
    if (alive) alive = mbar_wait(&full[stage], (it / LD_STAGES) & 1, p.status, ST_TIMEOUT_FULL);
    const uint32_t kv = smem_u32(s_kv + stage * stage_bytes);
    // ---- scores of 16 keys, a quarter of the columns
    float sc[MT][2][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int e = 0; e < 8; ++e) sc[m][e >> 2][e & 3] = 0.f;
#pragma unroll 3
    for (int kk = k_lo; kk < k_hi; ++kk) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4(kv + ld_swz(LD_TILE, kg + (mat >> 1) * 8 + (lane & 7), kk * 2 + (mat & 1)), b0, b1, b2, b3);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        uint32_t a[4];
        ldsm_x4(q_base + ld_swz(HR, m * 16 + (mat & 1) * 8 + (lane & 7), kk * 2 + (mat >> 1)), a[0], a[1], a[2], a[3]);
        mma_bf16(sc[m][0], a, b0, b1);
        mma_bf16(sc[m][1], a, b2, b3);
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        float* d = s_s + (part * HR + m * 16 + g) * SLD + kg + n * 8 + q4 * 2;
        *reinterpret_cast<float2*>(d) = make_float2(sc[m][n][0], sc[m][n][1]);
        *reinterpret_cast<float2*>(d + 8 * SLD) = make_float2(sc[m][n][2], sc[m][n][3]);
      }
    group_sync();
    // ---- softmax of one head row by TPR threads
    {
      const int row0 = (tile0 + grp + it * LD_GROUPS) * LD_TILE;
      const int valid = ctx - row0, hidden = first - row0;         // keys of this tile that exist; that lie before the window
      float v[KPT];
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        float s = 0.f;
#pragma unroll
        for (int x = 0; x < LD_PARTS; ++x) s += s_s[(x * HR + srow) * SLD + sk0 + i];
        v[i] = sk0 + i < valid && sk0 + i >= hidden ? s * scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int x = 1; x < TPR; x <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
      const float mn = fmaxf(m_run, mx);                           // a tile has at least one visible key
      const float cor = exp2f(m_run - mn);
      m_run = mn;
      float rs = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        const float e0 = exp2f(v[i] - mn), e1 = exp2f(v[i + 1] - mn);
        rs += e0 + e1;
        const int key = sk0 + i;
        *reinterpret_cast<uint32_t*>(s_p + ld_swz(HR, srow, key >> 3) + (key & 7) * 2) = pack_bf16(e0, e1);
      }
      l_run = l_run * cor + rs;
      if (gt % TPR == 0) s_cor[srow] = cor;
    }
    group_sync();
    // ---- O = O * cor + P V
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float c0 = s_cor[m * 16 + g], c1 = s_cor[m * 16 + g + 8];
      if (c0 == 1.f && c1 == 1.f) continue;
#pragma unroll
      for (int n = 0; n < NPW; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          o[m][n][e][0] *= c0;
          o[m][n][e][1] *= c0;
          o[m][n][e][2] *= c1;
          o[m][n][e][3] *= c1;
        }
    }
#pragma unroll
    for (int ks = 0; ks < LD_TILE / 16; ++ks) {
      uint32_t a[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
        ldsm_x4(p_base + ld_swz(HR, m * 16 + (mat & 1) * 8 + (lane & 7), ks * 2 + (mat >> 1)), a[m][0], a[m][1], a[m][2],
                a[m][3]);
#pragma unroll
      for (int n = 0; n < NPW; ++n) {
        const int cg = warp + n * LD_WARPS;                        // 16-column group of the latent
        if (cg * 16 >= p.V) continue;
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(kv + ld_swz(LD_TILE, ks * 16 + (mat & 1) * 8 + (lane & 7), cg * 2 + (mat >> 1)), b0, b1, b2, b3);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16(o[m][n][0], a[m], b0, b1);
          mma_bf16(o[m][n][1], a[m], b2, b3);
        }
      }
    }
    group_sync();                                                  // every warp is done with this stage, S and P
    if (gt == 0 && alive && it + LD_STAGES < n_mine) load_tile(it + LD_STAGES);
  }
  // ---- merge the groups: group 1 leaves its accumulators, maxima and sums in shared memory, group 0 combines and writes
#pragma unroll
  for (int x = 1; x < TPR; x <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, x);
  __syncthreads();
  float* s_o = reinterpret_cast<float*>(s_all);                    // [value of a thread][thread of the group]
  if (grp == 1) {
    if (gt % TPR == 0) {
      s_m[srow] = m_run;
      s_m[HR + srow] = l_run;
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < NPW; ++n)
#pragma unroll
        for (int e = 0; e < 8; ++e) s_o[((m * NPW + n) * 8 + e) * LD_GT + gt] = o[m][n][e >> 2][e & 3];
  }
  __syncthreads();
  if (grp == 1) return;
  float* s_w = s_cor;                                              // [2][HR] weight / sum of the two groups
  if (gt % TPR == 0) {
    const float m1 = s_m[srow], mm = fmaxf(m_run, m1);
    const float w0 = m_run == -INFINITY ? 0.f : exp2f(m_run - mm), w1 = m1 == -INFINITY ? 0.f : exp2f(m1 - mm);
    float l = l_run * w0 + s_m[HR + srow] * w1;
    const int head = h0 + srow;
    if (p.splits > 1 && head < p.H)
      p.part_lse[((long long)t * p.H + head) * p.splits + split] = l > 0.f ? mm + log2f(l) : -INFINITY;
    if (p.splits == 1 && p.sink != nullptr && head < p.H && l > 0.f) l += exp2f(p.sink[head] * 1.4426950408889634f - mm);
    float inv = l > 0.f ? 1.f / l : 0.f;
    if (p.splits == 1 && p.head_gate != nullptr && head < p.H) inv *= p.head_gate[(long long)t * p.H + head];
    s_w[srow] = w0 * inv;
    s_w[HR + srow] = w1 * inv;
  }
  group_sync();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = m * 16 + half * 8 + g;
      if (h0 + r >= p.H) continue;
      const float w0 = s_w[r], w1 = s_w[HR + r];
      const long long row = (long long)t * p.H + h0 + r;
#pragma unroll
      for (int n = 0; n < NPW; ++n) {
        const int cg = warp + n * LD_WARPS;
        if (cg * 16 >= p.V) continue;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int col = cg * 16 + e * 8 + q4 * 2, i0 = (m * NPW + n) * 8 + e * 4 + half * 2;
          const float a = o[m][n][e][half * 2] * w0 + s_o[i0 * LD_GT + gt] * w1;
          const float c = o[m][n][e][half * 2 + 1] * w0 + s_o[(i0 + 1) * LD_GT + gt] * w1;
          if (p.splits == 1)
            *reinterpret_cast<uint32_t*>(reinterpret_cast<bf16*>(p.out) + t * p.ld_out + (h0 + r) * p.V + col) = pack_bf16(a, c);
          else
            *reinterpret_cast<float2*>(p.part_o + (row * p.splits + split) * p.V + col) = make_float2(a, c);
        }
      }
    }
}
// out[row] = sum_s 2^(lse_s - max) part_o[row, s] / (sum_s 2^(lse_s - max) + sink); one CTA per (row, head), 4 columns a thread
__global__ void __launch_bounds__(128)
latent_merge_kernel(const RowAttn p) {
  __shared__ float s_w[LD_MAX_SPLITS];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x, t = row / p.H;
  const int h = int(row - t * p.H);
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    const float l = lane < p.splits ? __ldcg(p.part_lse + row * p.splits + lane) : -INFINITY;
    const float mx = warp_max(l);
    const float wgt = l == -INFINITY ? 0.f : exp2f(l - mx);
    float den = warp_sum(wgt);
    if (p.sink != nullptr && den > 0.f) den += exp2f(p.sink[h] * 1.4426950408889634f - mx);
    const float f = p.head_gate != nullptr ? p.head_gate[row] : 1.f;
    s_w[lane] = den > 0.f ? wgt / den * f : 0.f;
  }
  __syncthreads();
  for (int c = threadIdx.x * 4; c < p.V; c += 512) {
    float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) {
      const float f = s_w[s];
      const float4 v = __ldcg(reinterpret_cast<const float4*>(p.part_o + (row * p.splits + s) * p.V + c));
      a[0] = fmaf(f, v.x, a[0]);
      a[1] = fmaf(f, v.y, a[1]);
      a[2] = fmaf(f, v.z, a[2]);
      a[3] = fmaf(f, v.w, a[3]);
    }
    store4(reinterpret_cast<bf16*>(p.out) + t * p.ld_out + h * p.V + c, a[0], a[1], a[2], a[3]);
  }
}
void launch_latent_merge(const RowAttn& p, cudaStream_t s) {
  launch_pdl(PDL_DECODE_MERGE, latent_merge_kernel, dim3(unsigned((long long)p.T * p.H)), dim3(128), 0, s, p);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("latent merge: ") + cudaGetErrorString(e));
}

static int ld_box_rows(int block_size) {
  int box = LD_TILE;
  while (box > block_size || block_size % box != 0) box >>= 1;
  return box;
}
static int ld_nc(const RowAttn& p) { return (p.row_width + 63) / 64; }
static int ld_smem(int mt, int nc) {
  const int hr = mt * 16;
  return LD_GROUPS * LD_STAGES * nc * LD_SUB + nc * hr * 128 + LD_GROUPS * hr * 128 +
         LD_GROUPS * LD_PARTS * hr * (LD_TILE + 4) * 4 + (2 + LD_GROUPS) * hr * 4 + LD_GROUPS * LD_STAGES * 8 + 1024;
}
static int ld_mt(const RowAttn& p) {
  int mt = p.H > 32 ? 4 : p.H > 16 ? 2 : 1;
  while (mt > 1 && (ld_smem(mt, ld_nc(p)) > 227 * 1024 || (mt == 4 && p.V > 256))) mt >>= 1;
  return mt;
}

bool latent_decode_supported(const RowAttn& p) {
  return p.v_col == 0 && p.v_heads == 1 && p.V % 16 == 0 && p.V <= 512 && p.K % 8 == 0 && p.ld_out % 4 == 0 && ld_box_rows(p.block_size) >= 8 &&
         ld_smem(ld_mt(p), ld_nc(p)) <= 227 * 1024;
}

int latent_decode_splits(const RowAttn& p, int max_ctx, int num_sms) {
  const int hr = ld_mt(p) * 16;
  const int ctas = p.T * ((p.H + hr - 1) / hr);
  const int by_len = std::max(1, max_ctx / (4 * LD_TILE));      // two tiles per group at least
  int s = std::max(1, std::min({num_sms / std::max(1, ctas), by_len, LD_MAX_SPLITS}));
  if (ctas < num_sms && ctas * 3 > num_sms * 2) s = 1;             // nearly a full wave already
  return s;
}

void launch_latent_decode(const RowAttn& p, cudaStream_t s) {
  if (p.T == 0) return;
  const int box = ld_box_rows(p.block_size), nc = ld_nc(p), mt = ld_mt(p), smem = ld_smem(mt, nc);
  const CUtensorMap tm = make_tmap_bf16_2d(p.pool, (uint64_t)p.num_blocks * p.block_size, p.row_width, p.row_width, box, 64);
  const dim3 grid(p.T, (p.H + mt * 16 - 1) / (mt * 16), p.splits);
  const float scale_log2 = p.scale * 1.4426950408889634f;
  auto go = [&](auto kern) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    // ordinary launch like the other paged decode attention
    launch_pdl(PDL_DECODE_ATTN, kern, grid, dim3(LD_THREADS), smem, s, tm, p, box, nc, scale_log2);
  };
  auto pick = [&](auto m) {
    constexpr int MT = decltype(m)::value;
    if (p.V <= 128) go(latent_decode_kernel<MT, 1>);
    else if (p.V <= 256) go(latent_decode_kernel<MT, 2>);
    else if constexpr (MT < 4) go(latent_decode_kernel<MT, 4>);    // ld_mt keeps the accumulators in registers
  };
  if (mt == 1) pick(std::integral_constant<int, 1>{});
  else if (mt == 2) pick(std::integral_constant<int, 2>{});
  else pick(std::integral_constant<int, 4>{});
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("latent decode: ") + cudaGetErrorString(e));
}

// ------------------------------------------------------------------ per-head products
// y[g][m, n] = sum_k x[g][m, k] w[g][n, k] for decode-size batches.  CTA: 64 rows n of w (the M side of mma.sync m16n8k16,
// 16 per warp, so that no row of the tensor-core tile is wasted on a small batch) x NT * 8 rows m of x; both operands
// come in 64-column steps through a three-stage cp.async ring.
constexpr int HL_N = 64, HL_K = 64, HL_STAGES = 3, HL_THREADS = 128;
template <int NT>
__global__ void __launch_bounds__(HL_THREADS)
head_linear_kernel(const SimtLinear a) {
  constexpr int XR = NT * 8;                                       // rows of x
  __shared__ __align__(128) uint8_t s_w[HL_STAGES][HL_N * 128], s_x[HL_STAGES][XR * 128];
  pdl_launch_dependents();
  const int g = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n0 = blockIdx.x * HL_N, m0 = blockIdx.z * XR;
  const bf16* w = reinterpret_cast<const bf16*>(a.w) + g * a.gw;
  const bf16* x = reinterpret_cast<const bf16*>(a.x) + g * a.gx;
  const int steps = (a.K + HL_K - 1) / HL_K;
  auto load = [&](int st, bool wpart, bool xpart) {
    const int k0 = st * HL_K;
    if (wpart)
      for (int i = tid; i < HL_N * 8; i += HL_THREADS) {
        const int r = i >> 3, c = i & 7;
        const bool ok = n0 + r < a.N && k0 + c * 8 < a.K;
        cp_async16(smem_u32(s_w[st % HL_STAGES]) + r * 128 + ((c ^ (r & 7)) << 4),
                   ok ? w + (long long)(n0 + r) * a.ldw + k0 + c * 8 : w, ok);
      }
    if (xpart)
      for (int i = tid; i < XR * 8; i += HL_THREADS) {
        const int r = i >> 3, c = i & 7;
        const bool ok = m0 + r < a.M && k0 + c * 8 < a.K;
        cp_async16(smem_u32(s_x[st % HL_STAGES]) + r * 128 + ((c ^ (r & 7)) << 4),
                   ok ? x + (long long)(m0 + r) * a.ldx + k0 + c * 8 : x, ok);
      }
  };
  load(0, true, false);                                            // weights do not depend on the kernel before
  if (steps > 1) load(1, true, false);
  pdl_wait();
  load(0, false, true);
  cp_async_commit();
  if (steps > 1) load(1, false, true);
  cp_async_commit();
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const int mat = lane >> 3;
  for (int st = 0; st < steps; ++st) {
    cp_async_wait<1>();
    __syncthreads();
    if (st + 2 < steps) load(st + 2, true, true);
    cp_async_commit();
    const uint32_t ws = smem_u32(s_w[st % HL_STAGES]), xs = smem_u32(s_x[st % HL_STAGES]);
#pragma unroll
    for (int kk = 0; kk < HL_K / 16; ++kk) {
      uint32_t af[4];
      {
        const int r = warp * 16 + (mat & 1) * 8 + (lane & 7), c = kk * 2 + (mat >> 1);
        ldsm_x4(ws + r * 128 + ((c ^ (r & 7)) << 4), af[0], af[1], af[2], af[3]);
      }
#pragma unroll
      for (int i = 0; i < NT; i += 2) {
        uint32_t b0, b1, b2, b3;
        const int r = min(i * 8 + (mat >> 1) * 8 + (lane & 7), XR - 1), c = kk * 2 + (mat & 1);
        ldsm_x4(xs + r * 128 + ((c ^ (r & 7)) << 4), b0, b1, b2, b3);
        mma_bf16(acc[i], af, b0, b1);
        if (i + 1 < NT) mma_bf16(acc[i + 1], af, b2, b3);
      }
    }
  }
  // through shared memory, so that a row of y is written (and its gate read) 16 bytes at a time
  __syncthreads();
  constexpr int YP = HL_N + 8;
  static_assert(XR * YP * 2 <= int(sizeof(s_w)), "staging fits the weight ring");
  bf16* s_y = reinterpret_cast<bf16*>(&s_w[0][0]);
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      s_y[(i * 8 + (lane & 3) * 2 + (e & 1)) * YP + warp * 16 + (lane >> 2) + (e >> 1) * 8] = __float2bfloat16(acc[i][e]);
  __syncthreads();
  bf16* y = reinterpret_cast<bf16*>(a.y) + g * a.gy;
  const bf16* gate = reinterpret_cast<const bf16*>(a.gate.p);
  for (int i = tid; i < XR * (HL_N / 8); i += HL_THREADS) {
    const int m = i / (HL_N / 8), n = (i % (HL_N / 8)) * 8;
    if (m0 + m >= a.M || n0 + n >= a.N) continue;                  // N is a multiple of 8
    uint4 u = *reinterpret_cast<const uint4*>(s_y + m * YP + n);
    if (gate != nullptr) {
      const uint4 gu = __ldcg(reinterpret_cast<const uint4*>(gate + (long long)(m0 + m) * a.gate.ld + a.gate_off + g * a.N +
                                                             n0 + n));
      uint32_t uw[4] = {u.x, u.y, u.z, u.w};
      const uint32_t gw[4] = {gu.x, gu.y, gu.z, gu.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&uw[e]));
        const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[e]));
        uw[e] = pack_bf16(v.x * sigmoid_t<bf16>(q.x), v.y * sigmoid_t<bf16>(q.y));
      }
      u = make_uint4(uw[0], uw[1], uw[2], uw[3]);
    }
    *reinterpret_cast<uint4*>(y + (long long)(m0 + m) * a.ldy + n0 + n) = u;
  }
  const int pad = a.y_pad - a.groups * a.N;
  if (pad > 0 && g == 0 && blockIdx.x == 0)
    for (int i = tid; i < XR * pad; i += HL_THREADS)
      if (m0 + i / pad < a.M)
        reinterpret_cast<bf16*>(a.y)[(long long)(m0 + i / pad) * a.ldy + a.groups * a.N + i % pad] = __float2bfloat16(0.f);
}

bool head_linear_mma_supported(const SimtLinear& a) {
  if (a.N % 8 != 0 || a.ldy % 8 != 0 || a.gy % 8 != 0 || a.gate.part != nullptr) return false;
  if (a.gate.p != nullptr && (a.gate.ld % 8 != 0 || a.gate_off % 8 != 0)) return false;
  return a.K % 8 == 0 && a.ldx % 8 == 0 && a.ldw % 8 == 0 && a.gx % 8 == 0 && a.gw % 8 == 0 && a.bias == nullptr;
}
void launch_head_linear_mma(const SimtLinear& a, cudaStream_t s) {
  if (a.M == 0 || a.N == 0) return;
  auto go = [&](auto kern, int rows) {
    launch_pdl(PDL_SKINNY_GEMM, kern, dim3((a.N + HL_N - 1) / HL_N, a.groups, (a.M + rows - 1) / rows), dim3(HL_THREADS), 0,
               s, a);
  };
  if (a.M <= 8) go(head_linear_kernel<1>, 8);
  else if (a.M <= 32) go(head_linear_kernel<4>, 32);
  else go(head_linear_kernel<8>, 64);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("per-head product: ") + cudaGetErrorString(e));
}

}  // namespace fc
