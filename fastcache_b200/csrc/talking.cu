// Attention whose heads mix their scores before the softmax (talking heads), around the cache: rotation, norm per head, store of
// the cache rows, and the mix.  Scores are linear in the query, so the mix moves there: the score of head h with a key row is
//     sum_g talk[h, g] q_g . k_u(g) = sum_u (sum_{g of u} talk[h, g] q_g) . k_u,
// an ordinary product of a query as wide as the keys of all key heads together with a cache row that holds them side by side.
// The attention itself is that of rows shared by all heads (latent.cu, latent_decode*.cu, latent_prefill.cu).
#include <algorithm>
#include <stdexcept>
#include <string>

#include "hybrid.cuh"
#include "launch.h"
#include "mma.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int TS_BLOCK = 8;          // heads of the mix per thread and pass

// `tokens` consecutive tokens per CTA.  The projections are staged in shared memory as fp32, a warp rotates and norms a head
// there, then a thread makes TS_BLOCK heads of one column (PAIR: of two) of the mixed queries.
template <typename T, int THREADS, bool PAIR>
__global__ void __launch_bounds__(THREADS)
talk_store_kernel(const TalkStore p, int tokens) {
  extern __shared__ __align__(16) float sm[];
  const int H = p.H, G = p.G, D = p.D, V = p.V, nq = H * D, nk = G * D, nv = G * V, half = p.rot_dims / 2;
  const int per = H / G, hp = (H + TS_BLOCK - 1) / TS_BLOCK * TS_BLOCK;
  float* s_talk = sm;                                        // [g][hp]: transposed
  float* s_q = s_talk + H * hp;                              // q | k
  float2* cs = reinterpret_cast<float2*>(s_q + (nq + nk + 1) / 2 * 2);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int i = tid; i < H * hp; i += THREADS) {
    const int g = i / hp, h = i - g * hp;
    s_talk[i] = h < H ? p.talk[h * H + g] : 0.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  const bool keys = p.off_k >= 0;
  const bool vec = p.off_q % 4 == 0 && (!keys || p.off_k % 4 == 0);
  const long long t1 = min((long long)p.T, (long long)(blockIdx.x + 1) * tokens);
  for (long long t = (long long)blockIdx.x * tokens; t < t1; ++t) {
    const double pos = double(p.positions[t]);
    if (t != (long long)blockIdx.x * tokens) __syncthreads();
    auto stage = [&](float* dst, int off, int n) {
      if (vec && n % 4 == 0) {
        for (int i = tid * 4; i < n; i += THREADS * 4) *reinterpret_cast<float4*>(dst + i) = proj_at4<T>(p.proj, t, off + i);
      } else {
        for (int i = tid; i < n; i += THREADS) dst[i] = proj_at<T>(p.proj, t, off + i);
      }
    };
    stage(s_q, p.off_q, nq);
    if (keys) {
      if (nq % 4 == 0) stage(s_q + nq, p.off_k, nk);
      else
        for (int i = tid; i < nk; i += THREADS) s_q[nq + i] = proj_at<T>(p.proj, t, p.off_k + i);
    }
    for (int i = tid; i < half; i += THREADS) {
      float c, s;
      turn_angle(pos, p.freq[i], c, s);
      cs[i] = make_float2(c, s);
    }
    T* out = reinterpret_cast<T*>(p.out);
    if (tid < p.pad_out) out[t * p.ld_out + H * V + tid] = Elem<T>::put(0.f);
    int slot = keys ? p.slots[t] : -1;
    if (slot >= p.num_rows) {
      if (tid == 0) report(p.status, ST_BAD_INDEX);
      slot = -1;
    }
    T* row = reinterpret_cast<T*>(p.pool) + (slot >= 0 ? (long long)slot * p.row_width : 0);
    if (slot >= 0)
      for (int i = tid; i < nv; i += THREADS) row[p.v_col + i] = Elem<T>::put(proj_at<T>(p.proj, t, p.off_v + i));
    __syncthreads();
    for (int h = warp; h < H + (keys ? G : 0); h += THREADS / 32) {
      float* x = s_q + h * D;
      float ss = 0.f;
      for (int c = lane; c < half; c += 32) {
        const float u = x[c], v = x[half + c];
        const float2 a = cs[c];
        const float nu = u * a.x - v * a.y, nv2 = v * a.x + u * a.y;
        x[c] = nu;
        x[half + c] = nv2;
        ss += nu * nu + nv2 * nv2;
      }
      for (int c = 2 * half + lane; c < D; c += 32) ss += x[c] * x[c];
      const float inv = rsqrtf(warp_sum(ss) / float(D) + p.eps);
      __syncwarp();
      if (h < H) {
        for (int c = lane; c < D; c += 32) x[c] *= inv;
      } else if (slot >= 0) {
        for (int c = lane; c < D; c += 32) row[(h - H) * D + c] = Elem<T>::put(x[c] * inv);
      }
    }
    __syncthreads();
    constexpr int W = PAIR ? 2 : 1;
    const int cols = nk / W;
    T* q = reinterpret_cast<T*>(p.q) + t * H * nk;
    for (int i = tid; i < cols * (hp / TS_BLOCK); i += THREADS) {
      const int b = i / cols, c = (i - b * cols) * W, h0 = b * TS_BLOCK, u = c / D;
      float acc[TS_BLOCK][W];
#pragma unroll
      for (int e = 0; e < TS_BLOCK; ++e)
#pragma unroll
        for (int w = 0; w < W; ++w) acc[e][w] = 0.f;
      const float* x = s_q + u * per * D + (c - u * D);
      const float* tk = s_talk + u * per * hp + h0;
#pragma unroll 4
      for (int g = 0; g < per; ++g, x += D, tk += hp) {
        float v[W];
        if constexpr (PAIR) {
          const float2 f = *reinterpret_cast<const float2*>(x);
          v[0] = f.x;
          v[1] = f.y;
        } else {
          v[0] = *x;
        }
        const float4 a = *reinterpret_cast<const float4*>(tk), d = *reinterpret_cast<const float4*>(tk + 4);
        const float f[TS_BLOCK] = {a.x, a.y, a.z, a.w, d.x, d.y, d.z, d.w};
#pragma unroll
        for (int e = 0; e < TS_BLOCK; ++e)
#pragma unroll
          for (int w = 0; w < W; ++w) acc[e][w] = fmaf(f[e], v[w], acc[e][w]);
      }
#pragma unroll
      for (int e = 0; e < TS_BLOCK; ++e) {
        if (h0 + e >= H) break;
        T* d = q + (long long)(h0 + e) * nk + c;
        if constexpr (PAIR && sizeof(T) == 2) {
          *reinterpret_cast<uint32_t*>(d) = pack_bf16(acc[e][0], acc[e][1]);
        } else {
#pragma unroll
          for (int w = 0; w < W; ++w) d[w] = Elem<T>::put(acc[e][w]);
        }
      }
    }
  }
}

// Many rows of a finished projection (bf16), heads of 32, 64 or 128 columns.  D / 4 lanes hold a head, rotate and norm it in
// registers and leave it in shared memory as the sum of two bf16 terms.  The mix runs on mma.sync with talk as the 16-row operand,
// also as two terms: hi hi + hi lo + lo hi.  Inside a block of 32 columns, column 8 q + 2 j + e lies at 8 j + 2 q + e, so that a
// lane's four pairs of accumulators are eight neighbouring columns.  The next token's heads are requested before this one's mix.
// NR: query heads per D / 4 lanes, at most
constexpr int TR_THREADS = 256, TR_WARPS = TR_THREADS / 32;
template <int D, int NR>
__global__ void __launch_bounds__(TR_THREADS, NR <= 4 ? 3 : 2)
talk_store_rows_kernel(const TalkStore p, int tokens) {
  constexpr int L = D / 4, PER_WARP = 32 / L, PITCH = D + 8;  // lanes per head; pitch: rows 16 bytes apart modulo 128
  extern __shared__ __align__(16) uint8_t raw[];
  const int H = p.H, G = p.G, V = p.V, per = H / G, hp = (H + 15) / 16 * 16, kp = (per + 15) / 16 * 16, tp = kp + 8, half = p.rot_dims / 2;
  bf16* s_talk = reinterpret_cast<bf16*>(raw);               // [2][G][hp][tp]
  bf16* s_q = s_talk + 2 * G * hp * tp;                      // [2][H + 16][PITCH]
  float2* s_cs = reinterpret_cast<float2*>(s_q + 2 * (H + 16) * PITCH);      // [2][half]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  auto low = [](float v, bf16 hi) { return __float2bfloat16(v - __bfloat162float(hi)); };
  for (int i = tid; i < G * hp * tp; i += TR_THREADS) {
    const int u = i / (hp * tp), h = i / tp - u * hp, k = i % tp;
    const float v = h < H && k < per ? p.talk[h * H + u * per + k] : 0.f;
    const bf16 hi = __float2bfloat16(v);
    s_talk[i] = hi;
    s_talk[G * hp * tp + i] = low(v, hi);
  }
  for (int i = tid; i < 2 * 16 * PITCH; i += TR_THREADS) {   // rows behind the last head: read with zero weights
    const int part = i / (16 * PITCH);
    s_q[(part * (H + 16) + H) * PITCH + i - part * 16 * PITCH] = __float2bfloat16(0.f);
  }
  pdl_launch_dependents();
  pdl_wait();
  const bf16* src = reinterpret_cast<const bf16*>(p.proj.p);
  const bool keys = p.off_k >= 0;
  const int nk = G * D, t0 = blockIdx.x * tokens, t1 = min(p.T, t0 + tokens);
  const int sub = lane / L, l = lane - sub * L, c0 = l * 4;  // this lane's columns of a head
  const int at0 = (c0 & ~31) + ((c0 >> 1) & 3) * 8 + ((c0 >> 3) & 3) * 2;    // where the first of its two pairs lies (the other 8 behind)
  auto angles = [&](int t) {
    if (t < t1 && tid < half) {
      float c, s;
      turn_angle(double(p.positions[t]), p.freq[tid], c, s);
      s_cs[(t & 1) * half + tid] = make_float2(c, s);
    }
  };
  angles(t0);
  const int mat = lane >> 3;
  const uint32_t talk_u = smem_u32(s_talk), q_u = smem_u32(s_q);
  const uint32_t talk_lo = uint32_t(G * hp * tp) * 2, q_lo = uint32_t((H + 16) * PITCH) * 2;
  // one head per round: query heads, then (round NR) key heads
  auto head_of = [&](int r) {
    const int i = (r < NR ? r * TR_WARPS + warp : warp) * PER_WARP + sub;
    return r < NR ? (i < H ? i : -1) : keys && i < G ? H + i : -1;
  };
  uint2 in[NR + 1];
  uint4 val = make_uint4(0, 0, 0, 0);
  int next_slot = -1;
  auto request = [&](int t) {
    const bf16* row = src + (long long)t * p.proj.ld;
#pragma unroll
    for (int r = 0; r <= NR; ++r) {
      const int h = head_of(r);
      in[r] = h < 0 ? make_uint2(0, 0)
                    : __ldcg(reinterpret_cast<const uint2*>(row + (h < H ? p.off_q + h * D : p.off_k + (h - H) * D) + c0));
    }
    if (keys) {
      if (tid * 8 < G * V) val = __ldcg(reinterpret_cast<const uint4*>(row + p.off_v + tid * 8));
      next_slot = p.slots[t];
    }
  };
  if (t0 < t1) request(t0);
  for (int t = t0; t < t1; ++t) {
    __syncthreads();                                         // angles are there, the mix of the token before is done
    const float2* cs = s_cs + (t & 1) * half;
    int slot = next_slot;
    if (slot >= p.num_rows) {
      if (tid == 0) report(p.status, ST_BAD_INDEX);
      slot = -1;
    }
    bf16* dst = reinterpret_cast<bf16*>(p.pool) + (slot >= 0 ? (long long)slot * p.row_width : 0);
#pragma unroll
    for (int r = 0; r <= NR; ++r) {
      const int h = head_of(r);
      const bool on = h >= 0 && (h < H || slot >= 0);
      const uint2 raw2 = in[r];
      float x[4] = {__uint_as_float(raw2.x << 16), __uint_as_float(raw2.x & 0xffff0000u), __uint_as_float(raw2.y << 16),
                    __uint_as_float(raw2.y & 0xffff0000u)};
      if (half > 0) {
        const bool lo = c0 < half, turn = c0 < 2 * half;
        const int from = turn ? (lo ? lane + half / 4 : lane - half / 4) : lane;
        const float f = lo ? -1.f : 1.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float o = __shfl_sync(0xffffffffu, x[e], from);
          if (turn) {
            const float2 a = cs[(lo ? c0 : c0 - half) + e];
            x[e] = x[e] * a.x + f * o * a.y;
          }
        }
      }
      float ss = x[0] * x[0] + x[1] * x[1] + x[2] * x[2] + x[3] * x[3];
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float inv = rsqrtf(ss / float(D) + p.eps);
      if (!on) continue;
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] *= inv;
      const uint32_t a = pack_bf16(x[0], x[1]), b = pack_bf16(x[2], x[3]);
      if (h < H) {
        const uint32_t la = pack_bf16(x[0] - __uint_as_float(a << 16), x[1] - __uint_as_float(a & 0xffff0000u));
        const uint32_t lb = pack_bf16(x[2] - __uint_as_float(b << 16), x[3] - __uint_as_float(b & 0xffff0000u));
        uint32_t* d = reinterpret_cast<uint32_t*>(s_q + h * PITCH + at0);
        d[0] = a;
        d[4] = b;
        d += (H + 16) * PITCH / 2;
        d[0] = la;
        d[4] = lb;
      } else {
        *reinterpret_cast<uint2*>(dst + (h - H) * D + c0) = make_uint2(a, b);
      }
    }
    if (slot >= 0 && tid * 8 < G * V) *reinterpret_cast<uint4*>(dst + p.v_col + tid * 8) = val;
    if (t + 1 < t1) request(t + 1);
    __syncthreads();
    angles(t + 1);
    bf16* q = reinterpret_cast<bf16*>(p.q) + (long long)t * H * nk;
    const int blocks = nk / 32, units = blocks * (hp / 16);
    for (int un = warp; un < units; un += TR_WARPS) {
      const int m = un / blocks, blk = un - m * blocks, u = blk * 32 / D, col = blk * 32 - u * D;
      float acc[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
      for (int ks = 0; ks < kp; ks += 16) {
        uint32_t ah[4], al[4];
        const uint32_t ta = talk_u + uint32_t(((u * hp + m * 16 + (mat & 1) * 8 + (lane & 7)) * tp + ks + (mat >> 1) * 8) * 2);
        ldsm_x4(ta, ah[0], ah[1], ah[2], ah[3]);
        ldsm_x4(ta + talk_lo, al[0], al[1], al[2], al[3]);
#pragma unroll
        for (int jj = 0; jj < 2; ++jj) {
          const uint32_t qa = q_u + uint32_t(((u * per + ks + (mat & 1) * 8 + (lane & 7)) * PITCH + col + jj * 16 + (mat >> 1) * 8) * 2);
          uint32_t b0, b1, b2, b3, d0, d1, d2, d3;
          ldsm_x4_t(qa, b0, b1, b2, b3);
          ldsm_x4_t(qa + q_lo, d0, d1, d2, d3);
          mma_bf16(acc[2 * jj], ah, b0, b1);
          mma_bf16(acc[2 * jj + 1], ah, b2, b3);
          mma_bf16(acc[2 * jj], ah, d0, d1);
          mma_bf16(acc[2 * jj + 1], ah, d2, d3);
          mma_bf16(acc[2 * jj], al, b0, b1);
          mma_bf16(acc[2 * jj + 1], al, b2, b3);
        }
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int h = m * 16 + r * 8 + (lane >> 2);
        if (h < H)
          *reinterpret_cast<uint4*>(q + (long long)h * nk + blk * 32 + (lane & 3) * 8) =
              make_uint4(pack_bf16(acc[0][2 * r], acc[0][2 * r + 1]), pack_bf16(acc[1][2 * r], acc[1][2 * r + 1]),
                         pack_bf16(acc[2][2 * r], acc[2][2 * r + 1]), pack_bf16(acc[3][2 * r], acc[3][2 * r + 1]));
      }
    }
  }
}
static size_t talk_rows_smem(const TalkStore& p) {
  const int hp = (p.H + 15) / 16 * 16, tp = (p.H / p.G + 15) / 16 * 16 + 8;
  return size_t(2) * p.G * hp * tp * 2 + size_t(2) * (p.H + 16) * (p.D + 8) * 2 + size_t(2) * p.rot_dims / 2 * 8;
}
static bool talk_rows_supported(const TalkStore& p) {
  const int half = p.rot_dims / 2;
  return p.T > 296 && p.proj.part == nullptr && (p.D == 32 || p.D == 64 || p.D == 128) && half % 4 == 0 && half <= TR_THREADS &&
         (p.G * p.V) % 8 == 0 && p.proj.ld % 8 == 0 && p.off_q % 8 == 0 && (p.off_k < 0 || (p.off_k % 8 == 0 && p.off_v % 8 == 0)) &&
         p.v_col % 8 == 0 && p.row_width % 8 == 0 && p.pad_out == 0 && talk_rows_smem(p) <= 100 * 1024 &&
         p.H <= 8 * TR_WARPS * (128 / p.D) && p.G <= TR_WARPS * (128 / p.D) && p.G * p.V <= TR_THREADS * 8;
}
static void launch_talk_rows(const TalkStore& p, cudaStream_t s) {
  const size_t smem = talk_rows_smem(p);
  const int tokens = std::max(1, (p.T + 148 * 3 - 1) / (148 * 3));
  auto go = [&](auto kern) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    launch_pdl(PDL_ROPE, kern, dim3((p.T + tokens - 1) / tokens), dim3(TR_THREADS), smem, s, p, tokens);
  };
  const bool few = p.H <= 4 * TR_WARPS * (128 / p.D);
  if (p.D == 32) few ? go(talk_store_rows_kernel<32, 4>) : go(talk_store_rows_kernel<32, 8>);
  else if (p.D == 64) few ? go(talk_store_rows_kernel<64, 4>) : go(talk_store_rows_kernel<64, 8>);
  else few ? go(talk_store_rows_kernel<128, 4>) : go(talk_store_rows_kernel<128, 8>);
}

template <typename T>
static void talk_store_t(const TalkStore& p, cudaStream_t s) {
  const int hp = (p.H + TS_BLOCK - 1) / TS_BLOCK * TS_BLOCK;
  const size_t smem = size_t(p.H * hp + (p.H * p.D + p.G * p.D + 1) / 2 * 2 + p.rot_dims) * 4;
  if (smem > 200 * 1024) throw std::runtime_error("mixed heads: query and key projections are limited to 40000 columns");
  auto go = [&](auto kern, int threads, int tokens) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    launch_pdl(PDL_ROPE, kern, dim3((p.T + tokens - 1) / tokens), dim3(threads), smem, s, p, tokens);
  };
  const bool pair = p.D % 2 == 0;
  if (p.T <= 296) {
    if (pair) go(talk_store_kernel<T, 512, true>, 512, 1);
    else go(talk_store_kernel<T, 512, false>, 512, 1);
  } else {
    const int tokens = std::max(1, std::min(8, p.T / (148 * 6)));
    if (pair) go(talk_store_kernel<T, 256, true>, 256, tokens);
    else go(talk_store_kernel<T, 256, false>, 256, tokens);
  }
}
void launch_talk_store(const TalkStore& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (f32) talk_store_t<float>(p, s);
  else if (talk_rows_supported(p)) launch_talk_rows(p, s);
  else talk_store_t<bf16>(p, s);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("mix of the heads and store: ") + cudaGetErrorString(e));
}

}  // namespace fc
