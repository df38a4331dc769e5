// Recurrent layers over long runs (bf16 models): chunks of 64 rows, products on the tensor cores.
//
// With S the state before a chunk and b the decay accumulated inside it, the recurrences have the form
//     U = U0 - W S,   O = Q' S + P U,   S <- diag(dec) S + K'^T U
//   gated linear attention: U = V, no W, b per key channel:
//       Q' = q e^b,  K' = k e^(b_end - b),  P_ij = sum_d q_id k_jd e^(b_id - b_jd) for j <= i,  dec = e^b_end
//   gated delta rule (b per head): the writes of a chunk depend on one another through the unit lower triangular
//       I + L, L_ij = beta_i e^(b_i - b_j) k_i.k_j for j < i; W and U0 solve (I + L) [W | U0] = diag(beta) [e^b k | v]
//       (Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"), P_ij = e^(b_i - b_j) q_i.k_j
//   matrix memory: U = [V | 1] (the last column is the normaliser), no W.  With log gates f (summed to b) and i, running
//       maximum m, c_j = i_j - b_j and u_i = m_i - b_i = max(m_0, max_(j <= i) c_j) every exponent is at most 0:
//       Q' = q e^(m_0 - u_i),  K' = k e^(c_j - u_end),  P_ij = e^(c_j - u_i) q_i.k_j,  dec = e^(m_0 - u_end)
// The first kernel computes W, U0, Q', K', P and dec of every chunk in parallel (m_0 of a chunk comes from the gate kernel
// of recurrence.cu); the second walks the chunks of a run with S in registers.
//
// Everything that enters the recurrence stays 32-bit grade: a tensor-core operand is the sum of two bf16 terms
// (hi + lo) and a product hi hi + hi lo + lo hi, accumulated in fp32.  Operands of the second kernel are stored in the
// register layout of mma.sync m16n8k16's A fragment (1 KiB per 16 x 16 block: hi, then lo), ready to load.
#include <stdexcept>
#include <string>

#include "hybrid.cuh"
#include "mma.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int CK = 64;                 // rows per chunk
constexpr int CK_MAX_D = 128;
constexpr int CK_P = 10;               // lower-triangular 16 x 16 blocks of P

// scratch of one (chunk, head): fragments of Q', K', P, W, then U0 [64, V] and dec [Dp]
struct ChunkLayout {
  int kd;                              // 16-column blocks of the key dimension
  int q, k, p, w;                      // first fragment
  long long u, dec, bytes;             // byte offsets, total
};
__host__ __device__ inline ChunkLayout chunk_layout(int D, int V, bool delta) {
  ChunkLayout l;
  l.kd = (D + 15) / 16;
  l.q = 0;
  l.k = 4 * l.kd;
  l.p = 8 * l.kd;
  l.w = l.p + CK_P;
  const long long frags = l.w + (delta ? 4 * l.kd : 0);
  l.u = frags * 1024;
  l.dec = l.u + (delta ? (long long)CK * ((V + 3) / 4 * 4) * 4 : 0);
  l.bytes = (l.dec + l.kd * 64 + 255) / 256 * 256;
  return l;
}
bool chunk_supported(int D, int V) { return D % 2 == 0 && D <= CK_MAX_D && V % 2 == 0; }
long long chunk_scratch_bytes(const StepParams& p, int T, int kind) {
  return (long long)(T / CK + p.runs.B) * p.H * chunk_layout(p.D, p.V, kind == REC_DELTA).bytes;
}

__device__ __forceinline__ void split_pack(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16(a - f.x, b - f.y);
}
struct Frag {                          // hi and lo registers of an A (4) or B (2) operand
  uint32_t h[4], l[4];
};
__device__ __forceinline__ void mma3(float (&c)[4], const Frag& a, uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
  mma_bf16(c, a.l, bh0, bh1);
  mma_bf16(c, a.h, bl0, bl1);
  mma_bf16(c, a.h, bh0, bh1);
}
__device__ __forceinline__ void store_frag(uint8_t* unit, int f, int lane, const Frag& a) {
  uint4* d = reinterpret_cast<uint4*>(unit + (long long)f * 1024);
  d[lane] = make_uint4(a.h[0], a.h[1], a.h[2], a.h[3]);
  d[32 + lane] = make_uint4(a.l[0], a.l[1], a.l[2], a.l[3]);
}
__device__ __forceinline__ Frag load_frag(const uint8_t* unit, int f, int lane) {
  const uint4* s = reinterpret_cast<const uint4*>(unit + (long long)f * 1024);
  const uint4 h = __ldcg(s + lane), l = __ldcg(s + 32 + lane);
  Frag a;
  a.h[0] = h.x; a.h[1] = h.y; a.h[2] = h.z; a.h[3] = h.w;
  a.l[0] = l.x; a.l[1] = l.y; a.l[2] = l.z; a.l[3] = l.w;
  return a;
}
// accumulators of a 16 x 16 block (two n8 tiles) as an A fragment
__device__ __forceinline__ Frag acc_frag(const float (&c0)[4], const float (&c1)[4]) {
  Frag a;
  split_pack(c0[0], c0[1], a.h[0], a.l[0]);
  split_pack(c0[2], c0[3], a.h[1], a.l[1]);
  split_pack(c1[0], c1[1], a.h[2], a.l[2]);
  split_pack(c1[2], c1[3], a.h[3], a.l[3]);
  return a;
}
// row pitch (floats) of a [64][Dp] tile: 8 mod 32, so that the 8-byte fragment reads are free of bank conflicts
__host__ __device__ inline int chunk_pitch(int kd) { return (kd * 16 + 31) / 32 * 32 + 8; }

struct ChunkId {
  Run run;
  int n, row0;                         // rows of this chunk, first flat row
  uint8_t* unit;                       // scratch of (chunk, head)
};
__device__ __forceinline__ bool chunk_of(const StepParams& p, const ChunkLayout& l, int c, int h, int b, ChunkId& o) {
  o.run = get_run(p.runs, b);
  o.n = min(CK, o.run.len - c * CK);
  o.row0 = o.run.lo + c * CK;
  // floor(lo / 64) + b leaves room for ceil(len / 64) chunks before the next run's first
  o.unit = p.scratch + ((long long)(o.run.lo / CK + b + c) * p.H + h) * l.bytes;
  return o.run.slot >= 0 && o.n > 0;
}

constexpr int CA_THREADS = 256;

// blocks (I, J) of the lower triangle in order
__device__ __forceinline__ void tri_block(int idx, int& I, int& J) {
  I = idx >= 6 ? 3 : idx >= 3 ? 2 : idx >= 1 ? 1 : 0;
  J = idx - I * (I + 1) / 2;
}

// ------------------------------------------------------------------ first kernel, gated delta rule
__global__ void __launch_bounds__(CA_THREADS)
delta_chunk_prepare_kernel(const StepParams p) {
  extern __shared__ float sm[];
  const ChunkLayout lay = chunk_layout(p.D, p.V, true);
  const int pitch = chunk_pitch(lay.kd), Dp = lay.kd * 16;
  float* s_k = sm;                                  // [64][pitch]
  float* s_q = s_k + CK * pitch;                    // [64][pitch], later columns of U0
  float* s_l = s_q + CK * max(pitch, CA_THREADS / 2);   // L transposed: [column j][row i], 64 x 64
  float* s_g = s_l + CK * CK;                       // accumulated log decay
  float* s_beta = s_g + CK;
  float* s_lg = s_beta + CK;
  float* s_eg = s_lg + CK;                          // e^b of a row, e^(b_end - b)
  float* s_ek = s_eg + CK;
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  ChunkId id;
  if (!chunk_of(p, lay, blockIdx.x, h, blockIdx.z, id)) return;
  const int K = p.H / p.group, hk = h / p.group;
  if (tid < CK) {
    s_lg[tid] = tid < id.n ? p.log_g[(long long)(id.row0 + tid) * p.H + h] : 0.f;
    s_beta[tid] = tid < id.n ? p.beta[(long long)(id.row0 + tid) * p.H + h] : 0.f;
  }
#pragma unroll 4
  for (int r = warp; r < CK; r += CA_THREADS / 32)
    for (int c = lane * 2; c < Dp; c += 64) {
      float2 q = make_float2(0.f, 0.f), k = q;
      if (r < id.n && c < p.D) {
        const float* src = p.qk + ((long long)(id.row0 + r) * 2 * K + hk) * p.D + c;
        q = *reinterpret_cast<const float2*>(src);
        k = *reinterpret_cast<const float2*>(src + (long long)K * p.D);
      }
      *reinterpret_cast<float2*>(s_q + r * pitch + c) = q;
      *reinterpret_cast<float2*>(s_k + r * pitch + c) = k;
    }
  __syncthreads();
  if (tid < CK) {
    float g = 0.f;
    for (int j = 0; j <= tid; ++j) g += s_lg[j];
    s_g[tid] = g;
  }
  __syncthreads();
  const float g_end = s_g[CK - 1];
  if (tid < CK) {
    s_eg[tid] = expf(s_g[tid]);
    s_ek[tid] = expf(g_end - s_g[tid]);
  }
  __syncthreads();
  const int gr = lane >> 2, gc = (lane & 3) * 2;
  // L and P, block by block
  for (int idx = warp; idx < CK_P; idx += CA_THREADS / 32) {
    int I, J;
    tri_block(idx, I, J);
    float ak[2][4] = {}, aq[2][4] = {};
    for (int kk = 0; kk < lay.kd; ++kk) {
      auto row2 = [&](const float* base, int r, int c) { return *reinterpret_cast<const float2*>(base + r * pitch + kk * 16 + c); };
      Frag fk, fq;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int r = I * 16 + gr + (x & 1) * 8, c = gc + (x >> 1) * 8;
        const float2 kv = row2(s_k, r, c), qv = row2(s_q, r, c);
        split_pack(kv.x, kv.y, fk.h[x], fk.l[x]);
        split_pack(qv.x, qv.y, fq.h[x], fq.l[x]);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const float2 kv = row2(s_k, J * 16 + n * 8 + gr, gc + x * 8);
          split_pack(kv.x, kv.y, bh[x], bl[x]);
        }
        mma3(ak[n], fk, bh[0], bh[1], bl[0], bl[1]);
        mma3(aq[n], fq, bh[0], bh[1], bl[0], bl[1]);
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = I * 16 + gr + (e >> 1) * 8, j = J * 16 + n * 8 + gc + (e & 1);
        const float f = j <= i ? expf(s_g[i] - s_g[j]) : 0.f;
        aq[n][e] *= f;
        s_l[j * CK + i] = j < i ? s_beta[i] * f * ak[n][e] : 0.f;
      }
    store_frag(id.unit, lay.p + idx, lane, acc_frag(aq[0], aq[1]));
  }
  // Q' and K'^T fragments
  for (int f = warp; f < 8 * lay.kd; f += CA_THREADS / 32) {
    Frag a;
    if (f < 4 * lay.kd) {
      const int I = f / lay.kd, kk = f - I * lay.kd;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int r = I * 16 + gr + (x & 1) * 8, c = kk * 16 + gc + (x >> 1) * 8;
        const float e = s_eg[r];
        split_pack(s_q[r * pitch + c] * e, s_q[r * pitch + c + 1] * e, a.h[x], a.l[x]);
      }
      store_frag(id.unit, lay.q + f, lane, a);
    } else {
      const int m = (f - 4 * lay.kd) / 4, kt = (f - 4 * lay.kd) & 3;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = m * 16 + gr + (x & 1) * 8, r = kt * 16 + gc + (x >> 1) * 8;
        split_pack(s_k[r * pitch + d] * s_ek[r], s_k[(r + 1) * pitch + d] * s_ek[r + 1],
                   a.h[x], a.l[x]);
      }
      store_frag(id.unit, lay.k + f - 4 * lay.kd, lane, a);
    }
  }
  for (int d = tid; d < Dp; d += CA_THREADS) reinterpret_cast<float*>(id.unit + lay.dec)[d] = s_eg[CK - 1];
  __syncthreads();
  // forward substitution, one right-hand-side column per thread and 16 rows at a time: the first half of the CTA takes
  // the key columns (W, in place of k), the second half value columns (U0, in slots of the q tile)
  const int V4 = (p.V + 3) / 4 * 4;
  float* u0 = reinterpret_cast<float*>(id.unit + lay.u);
  const bf16* v = reinterpret_cast<const bf16*>(p.v) + (long long)id.row0 * p.H * p.V + h * p.V;
  constexpr int HALF = CA_THREADS / 2;              // >= CK_MAX_D
  const bool key = tid < HALF;
  float* col = key ? s_k + tid : s_q + tid - HALF;
  const int ld = key ? pitch : HALF;
  for (int c = key ? tid : tid - HALF; c < (key ? Dp : V4); c += HALF) {
#pragma unroll 1
    for (int I = 0; I < 4; ++I) {
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const int r = I * 16 + i;
        if (key) x[i] = col[r * ld] * s_eg[r];
        else x[i] = r < id.n && c < p.V ? __bfloat162float(v[(long long)r * p.H * p.V + c]) : 0.f;
        x[i] *= s_beta[r];
      }
#pragma unroll 2
      for (int j = 0; j < I * 16; ++j) {
        const float xj = col[j * ld];
        const float4* lc = reinterpret_cast<const float4*>(s_l + j * CK + I * 16);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float4 lv = lc[q];
          x[q * 4] = fmaf(-lv.x, xj, x[q * 4]);
          x[q * 4 + 1] = fmaf(-lv.y, xj, x[q * 4 + 1]);
          x[q * 4 + 2] = fmaf(-lv.z, xj, x[q * 4 + 2]);
          x[q * 4 + 3] = fmaf(-lv.w, xj, x[q * 4 + 3]);
        }
      }
#pragma unroll
      for (int j = 0; j < 16; ++j) {                // entries of L on and above the diagonal are zero
        const float4* lc = reinterpret_cast<const float4*>(s_l + (I * 16 + j) * CK + I * 16);
#pragma unroll
        for (int q = j / 4; q < 4; ++q) {
          const float4 lv = lc[q];
          const float xj = x[j];
          if (q * 4 > j) x[q * 4] = fmaf(-lv.x, xj, x[q * 4]);
          if (q * 4 + 1 > j) x[q * 4 + 1] = fmaf(-lv.y, xj, x[q * 4 + 1]);
          if (q * 4 + 2 > j) x[q * 4 + 2] = fmaf(-lv.z, xj, x[q * 4 + 2]);
          if (q * 4 + 3 > j) x[q * 4 + 3] = fmaf(-lv.w, xj, x[q * 4 + 3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        col[(I * 16 + i) * ld] = x[i];
        if (!key) u0[(I * 16 + i) * V4 + c] = x[i];
      }
    }
  }
  __syncthreads();
  for (int f = warp; f < 4 * lay.kd; f += CA_THREADS / 32) {
    const int I = f / lay.kd, kk = f - I * lay.kd;
    Frag a;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const float2 w = *reinterpret_cast<const float2*>(s_k + (I * 16 + gr + (x & 1) * 8) * pitch + kk * 16 + gc + (x >> 1) * 8);
      split_pack(w.x, w.y, a.h[x], a.l[x]);
    }
    store_frag(id.unit, lay.w + f, lane, a);
  }
}

// ------------------------------------------------------------------ first kernel, gated linear attention
__global__ void __launch_bounds__(CA_THREADS)
gla_chunk_prepare_kernel(const StepParams p) {
  extern __shared__ float sm[];
  const ChunkLayout lay = chunk_layout(p.D, p.V, false);
  const int pitch = chunk_pitch(lay.kd), Dp = lay.kd * 16;
  float* s_k = sm;                                  // [64][pitch]
  float* s_q = s_k + CK * pitch;
  float* s_b = s_q + CK * pitch;                    // accumulated decay, log2
  float* s_d = s_b + CK * pitch;                    // [4][16][18] diagonal blocks of P
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  ChunkId id;
  if (!chunk_of(p, lay, blockIdx.x, h, blockIdx.z, id)) return;
  const bf16* proj = reinterpret_cast<const bf16*>(p.proj.p);
  const bf16* zp = reinterpret_cast<const bf16*>(p.z);
#pragma unroll 4
  for (int r = warp; r < CK; r += CA_THREADS / 32)
    for (int c = lane * 2; c < Dp; c += 64) {
      float2 q = make_float2(0.f, 0.f), k = q, g = q;
      if (r < id.n && c < p.D) {
        auto two = [](const bf16* s) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(s)); };
        const bf16* row = proj + (long long)(id.row0 + r) * p.proj.ld + h * p.D + c;
        q = two(row + p.off_q);
        k = two(row + p.off_k);
        g = two(zp + (long long)(id.row0 + r) * p.ld_z + h * p.D + c);
        const float2 zb = *reinterpret_cast<const float2*>(p.z_bias + h * p.D + c);
        const float f = p.inv_tau * 1.4426950408889634f;
        g = make_float2(log_sigmoid_f(g.x + zb.x) * f, log_sigmoid_f(g.y + zb.y) * f);
      }
      *reinterpret_cast<float2*>(s_q + r * pitch + c) = make_float2(q.x * p.q_scale, q.y * p.q_scale);
      *reinterpret_cast<float2*>(s_k + r * pitch + c) = k;
      *reinterpret_cast<float2*>(s_b + r * pitch + c) = g;
    }
  __syncthreads();
  for (int c = tid; c < Dp; c += CA_THREADS) {
    float acc = 0.f;
#pragma unroll 1
    for (int r = 0; r < CK; r += 16) {
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) x[i] = s_b[(r + i) * pitch + c];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        acc += x[i];
        s_b[(r + i) * pitch + c] = acc;
      }
    }
    reinterpret_cast<float*>(id.unit + lay.dec)[c] = exp2f(acc);
  }
  __syncthreads();
  const int gr = lane >> 2, gc = (lane & 3) * 2;
  // P: both factors of a 16 x 16 block decayed to a common row, the row before block I or, on the diagonal, its first
  // row.  There the key factor grows with the decay inside the block; should that leave the range of the format, the
  // block is computed from the exact differences instead.
  for (int idx = warp; idx < CK_P; idx += CA_THREADS / 32) {
    int I, J;
    tri_block(idx, I, J);
    const float* ref = s_b + (I == J ? I * 16 : I * 16 - 1) * pitch;
    if (I == J) {
      bool far = false;
      for (int c = lane; c < Dp; c += 32) far |= ref[c] - s_b[(I * 16 + 15) * pitch + c] > 60.f;
      if (__any_sync(0xffffffffu, far)) {
        float* s_p = s_d + I * 16 * 18;
        for (int i = 0; i < 16; ++i)
          for (int j = 0; j < 16; ++j) {
            float a = 0.f;
            if (j <= i)
              for (int c = lane; c < Dp; c += 32) {
                const int x = (I * 16 + i) * pitch + c, y = (I * 16 + j) * pitch + c;
                a = fmaf(s_q[x] * exp2f(s_b[x] - s_b[y]), s_k[y], a);
              }
            a = warp_sum(a);
            if (lane == 0) s_p[i * 18 + j] = a;
          }
        __syncwarp();
        Frag a;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float* s = s_p + (gr + (x & 1) * 8) * 18 + gc + (x >> 1) * 8;
          split_pack(s[0], s[1], a.h[x], a.l[x]);
        }
        store_frag(id.unit, lay.p + idx, lane, a);
        continue;
      }
    }
    float acc[2][4] = {};
    for (int kk = 0; kk < lay.kd; ++kk) {
      Frag fq;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int r = (I * 16 + gr + (x & 1) * 8) * pitch, c = kk * 16 + gc + (x >> 1) * 8;
        const float2 q = *reinterpret_cast<const float2*>(s_q + r + c), b = *reinterpret_cast<const float2*>(s_b + r + c),
                     f = *reinterpret_cast<const float2*>(ref + c);
        split_pack(q.x * exp2f(b.x - f.x), q.y * exp2f(b.y - f.y), fq.h[x], fq.l[x]);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int r = (J * 16 + n * 8 + gr) * pitch, c = kk * 16 + gc + x * 8;
          const float2 k = *reinterpret_cast<const float2*>(s_k + r + c), b = *reinterpret_cast<const float2*>(s_b + r + c),
                       f = *reinterpret_cast<const float2*>(ref + c);
          split_pack(k.x * exp2f(f.x - b.x), k.y * exp2f(f.y - b.y), bh[x], bl[x]);
        }
        mma3(acc[n], fq, bh[0], bh[1], bl[0], bl[1]);
      }
    }
    if (I == J)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (n * 8 + gc + (e & 1) > gr + (e >> 1) * 8) acc[n][e] = 0.f;
    store_frag(id.unit, lay.p + idx, lane, acc_frag(acc[0], acc[1]));
  }
  for (int f = warp; f < 8 * lay.kd; f += CA_THREADS / 32) {
    Frag a;
    if (f < 4 * lay.kd) {
      const int I = f / lay.kd, kk = f - I * lay.kd;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int o = (I * 16 + gr + (x & 1) * 8) * pitch + kk * 16 + gc + (x >> 1) * 8;
        split_pack(s_q[o] * exp2f(s_b[o]), s_q[o + 1] * exp2f(s_b[o + 1]), a.h[x], a.l[x]);
      }
      store_frag(id.unit, lay.q + f, lane, a);
    } else {
      const int m = (f - 4 * lay.kd) / 4, kt = (f - 4 * lay.kd) & 3;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = m * 16 + gr + (x & 1) * 8, o = (kt * 16 + gc + (x >> 1) * 8) * pitch + d;
        const float end = s_b[(CK - 1) * pitch + d];
        split_pack(s_k[o] * exp2f(end - s_b[o]), s_k[o + pitch] * exp2f(end - s_b[o + pitch]), a.h[x], a.l[x]);
      }
      store_frag(id.unit, lay.k + f - 4 * lay.kd, lane, a);
    }
  }
}

// ------------------------------------------------------------------ first kernel, matrix memory
__global__ void __launch_bounds__(CA_THREADS)
memory_chunk_prepare_kernel(const StepParams p) {
  extern __shared__ float sm[];
  const ChunkLayout lay = chunk_layout(p.D, p.V, false);
  const int pitch = chunk_pitch(lay.kd), Dp = lay.kd * 16;
  float* s_k = sm;                                  // [64][pitch]
  float* s_q = s_k + CK * pitch;
  float* s_c = s_q + CK * pitch;                    // c_j, u_i
  float* s_u = s_c + CK;
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  ChunkId id;
  if (!chunk_of(p, lay, blockIdx.x, h, blockIdx.z, id)) return;
  const bf16* proj = reinterpret_cast<const bf16*>(p.proj.p);
  const float m0 = blockIdx.x == 0 ? p.m_0[(long long)blockIdx.z * p.H + h] : p.m_t[(long long)(id.row0 - 1) * p.H + h];
  if (warp == 0) {                                  // two rows per lane: sums of f, then running maxima of c
    float f[2], g[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int r = lane * 2 + x;
      const long long o = (long long)(id.row0 + r) * p.H + h;
      f[x] = r < id.n ? p.log_f[o] : 0.f;
      g[x] = r < id.n ? p.log_i[o] : -INFINITY;     // rows past the run write nothing
    }
    float b = f[0] + f[1];
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, b, d);
      if (lane >= d) b += y;
    }
    const float c0 = g[0] - (b - f[1]), c1 = g[1] - b;
    float u = fmaxf(c0, c1);
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, u, d);
      if (lane >= d) u = fmaxf(u, y);
    }
    const float before = __shfl_up_sync(0xffffffffu, u, 1);
    const float u0 = fmaxf(m0, lane > 0 ? fmaxf(before, c0) : c0);
    s_c[lane * 2] = c0;
    s_c[lane * 2 + 1] = c1;
    s_u[lane * 2] = u0;
    s_u[lane * 2 + 1] = fmaxf(u0, c1);
  }
#pragma unroll 4
  for (int r = warp; r < CK; r += CA_THREADS / 32)
    for (int c = lane * 2; c < Dp; c += 64) {
      float2 q = make_float2(0.f, 0.f), k = q;
      if (r < id.n && c < p.D) {
        auto two = [](const bf16* s) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(s)); };
        const bf16* row = proj + (long long)(id.row0 + r) * p.proj.ld + h * p.D + c;
        q = two(row + p.off_q);
        k = two(row + p.off_k);
      }
      *reinterpret_cast<float2*>(s_q + r * pitch + c) = make_float2(q.x * p.q_scale, q.y * p.q_scale);
      *reinterpret_cast<float2*>(s_k + r * pitch + c) = k;
    }
  __syncthreads();
  const float u_end = s_u[CK - 1];
  const int gr = lane >> 2, gc = (lane & 3) * 2;
  for (int idx = warp; idx < CK_P; idx += CA_THREADS / 32) {
    int I, J;
    tri_block(idx, I, J);
    float acc[2][4] = {};
    for (int kk = 0; kk < lay.kd; ++kk) {
      Frag fq;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float2 q = *reinterpret_cast<const float2*>(s_q + (I * 16 + gr + (x & 1) * 8) * pitch + kk * 16 + gc + (x >> 1) * 8);
        split_pack(q.x, q.y, fq.h[x], fq.l[x]);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        uint32_t bh[2];                             // a key is a bf16 value: no second term
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const float2 k = *reinterpret_cast<const float2*>(s_k + (J * 16 + n * 8 + gr) * pitch + kk * 16 + gc + x * 8);
          bh[x] = pack_bf16(k.x, k.y);
        }
        mma_bf16(acc[n], fq.l, bh[0], bh[1]);
        mma_bf16(acc[n], fq.h, bh[0], bh[1]);
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = I * 16 + gr + (e >> 1) * 8, j = J * 16 + n * 8 + gc + (e & 1);
        acc[n][e] = j <= i ? acc[n][e] * expf(s_c[j] - s_u[i]) : 0.f;
      }
    store_frag(id.unit, lay.p + idx, lane, acc_frag(acc[0], acc[1]));
  }
  for (int f = warp; f < 8 * lay.kd; f += CA_THREADS / 32) {
    Frag a;
    if (f < 4 * lay.kd) {
      const int I = f / lay.kd, kk = f - I * lay.kd;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int r = I * 16 + gr + (x & 1) * 8, o = r * pitch + kk * 16 + gc + (x >> 1) * 8;
        const float e = expf(m0 - s_u[r]);
        split_pack(s_q[o] * e, s_q[o + 1] * e, a.h[x], a.l[x]);
      }
      store_frag(id.unit, lay.q + f, lane, a);
    } else {
      const int m = (f - 4 * lay.kd) / 4, kt = (f - 4 * lay.kd) & 3;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = m * 16 + gr + (x & 1) * 8, r = kt * 16 + gc + (x >> 1) * 8;
        split_pack(s_k[r * pitch + d] * expf(s_c[r] - u_end), s_k[(r + 1) * pitch + d] * expf(s_c[r + 1] - u_end), a.h[x], a.l[x]);
      }
      store_frag(id.unit, lay.k + f - 4 * lay.kd, lane, a);
    }
  }
  for (int d = tid; d < Dp; d += CA_THREADS) reinterpret_cast<float*>(id.unit + lay.dec)[d] = expf(m0 - u_end);
}

// ------------------------------------------------------------------ second kernel
// CTA = (block of VB value columns, head, request), four warps.  Warp w owns rows 16 w .. 16 w + 15 of a chunk for U and
// O, and the 16-row blocks w, w + 4 of S in registers; S and U go through shared memory as hi / lo operands.  Matrix memory
// has one column more, V: its S is the normaliser, its U is 1 and its O goes to `den`.
constexpr int CB_THREADS = 128;

template <int KIND, int VB>
__global__ void __launch_bounds__(CB_THREADS, VB == 16 ? 3 : 2)
chunk_scan_kernel(const StepParams p) {
  constexpr bool DELTA = KIND == REC_DELTA, MEM = KIND == REC_MEMORY;
  constexpr int N8 = VB / 8;
  constexpr int PITCH = VB + 8;                     // bf16; rows an odd number of 16-byte units apart
  extern __shared__ uint8_t smem_raw[];
  const ChunkLayout lay = chunk_layout(p.D, p.V, DELTA);
  const int kd = lay.kd, Dp = kd * 16;
  bf16* s_sh = reinterpret_cast<bf16*>(smem_raw);   // [Dp][PITCH] state, hi
  bf16* s_sl = s_sh + Dp * PITCH;
  bf16* s_uh = s_sl + Dp * PITCH;                   // [64][PITCH]
  bf16* s_ul = s_uh + CK * PITCH;
  const int h = blockIdx.y, b = blockIdx.z, v0 = blockIdx.x * VB;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, gc = (lane & 3) * 2;
  const Run run = get_run(p.runs, b);
  if (run.slot < 0 || run.len <= 0) {
    for (int i = tid; i < run.len * VB; i += CB_THREADS)
      if (v0 + i % VB < p.V) p.o_raw[((long long)(run.lo + i / VB) * p.H + h) * p.V + v0 + i % VB] = 0.f;
      else if (MEM && v0 + i % VB == p.V) p.den[(long long)(run.lo + i / VB) * p.H + h] = p.m_t[(long long)(run.lo + i / VB) * p.H + h] = 0.f;
    return;
  }
  float* st = p.state + ((long long)run.slot * p.H + h) * p.D * p.V;
  float* ns = MEM ? p.nstate + ((long long)run.slot * p.H + h) * p.D : nullptr;
  float S[2][N8][4];
  auto state_io = [&](bool load) {
#pragma unroll
    for (int mi = 0; mi < 2; ++mi)
#pragma unroll
      for (int n = 0; n < N8; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int d = (warp + mi * 4) * 16 + gr + half * 8, v = v0 + n * 8 + gc;
          if (MEM && d < p.D && v == p.V) {
            if (load) S[mi][n][half * 2] = ns[d];
            else ns[d] = S[mi][n][half * 2];
          }
          if (d >= p.D || v >= p.V) continue;       // V is even: a pair of columns exists or not
          float2* s = reinterpret_cast<float2*>(st + (long long)d * p.V + v);
          if (load) {
            const float2 x = *s;
            S[mi][n][half * 2] = x.x;
            S[mi][n][half * 2 + 1] = x.y;
          } else {
            *s = make_float2(S[mi][n][half * 2], S[mi][n][half * 2 + 1]);
          }
        }
  };
#pragma unroll
  for (int mi = 0; mi < 2; ++mi)
#pragma unroll
    for (int n = 0; n < N8; ++n) S[mi][n][0] = S[mi][n][1] = S[mi][n][2] = S[mi][n][3] = 0.f;
  if (run.start > 0) state_io(true);
  auto put_state = [&]() {
#pragma unroll
    for (int mi = 0; mi < 2; ++mi) {
      if (warp + mi * 4 >= kd) continue;
#pragma unroll
      for (int n = 0; n < N8; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int o = ((warp + mi * 4) * 16 + gr + half * 8) * PITCH + n * 8 + gc;
          uint32_t hi, lo;
          split_pack(S[mi][n][half * 2], S[mi][n][half * 2 + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(s_sh + o) = hi;
          *reinterpret_cast<uint32_t*>(s_sl + o) = lo;
        }
    }
  };
  put_state();
  __syncthreads();
  const uint32_t a_sh = smem_u32(s_sh), a_sl = smem_u32(s_sl), a_uh = smem_u32(s_uh), a_ul = smem_u32(s_ul);
  // B fragments (k16 x n16) of a [rows][PITCH] tile
  const uint32_t b_off = uint32_t((((lane >> 3) & 1) * 8 + (lane & 7)) * PITCH + (lane >> 4) * 8) * 2;
  auto ld_b = [&](uint32_t base, int kk, int n2, uint32_t (&r)[4]) {
    ldsm_x4_t(base + b_off + uint32_t(kk * 16 * PITCH + n2 * 16) * 2, r[0], r[1], r[2], r[3]);
  };
  const int V4 = (p.V + 3) / 4 * 4;
  const int n_chunks = (run.len + CK - 1) / CK;
  const int i0 = warp * 16 + gr;                    // this thread's rows of a chunk: i0 and i0 + 8
  constexpr int MAX_KD = CK_MAX_D / 16;
  float u[N8][4];
  Frag fq[3], fw[3];
  // U0 (or V) of this thread's rows and the first fragments of a chunk
  auto fetch = [&](const ChunkId& id) {
#pragma unroll
    for (int n = 0; n < N8; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = i0 + half * 8, v = v0 + n * 8 + gc;
        float2 x = make_float2(0.f, 0.f);
        if (v < p.V) {
          if (DELTA)
            x = __ldcg(reinterpret_cast<const float2*>(reinterpret_cast<const float*>(id.unit + lay.u) + i * V4 + v));
          else if (i < id.n)
            x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(
                reinterpret_cast<const bf16*>(p.proj.p) + (long long)(id.row0 + i) * p.proj.ld + p.off_v + h * p.V + v));
        } else if (MEM && v == p.V && i < id.n) {
          x.x = 1.f;
        }
        u[n][half * 2] = x.x;
        u[n][half * 2 + 1] = x.y;
      }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      if (x >= kd) continue;
      fq[x] = load_frag(id.unit, lay.q + warp * kd + x, lane);
      if (DELTA) fw[x] = load_frag(id.unit, lay.w + warp * kd + x, lane);
    }
  };
  ChunkId id;
  chunk_of(p, lay, 0, h, b, id);
  fetch(id);
  for (int c = 0; c < n_chunks; ++c) {
    // ---- products with the state before the chunk: O = Q' S, U = U0 - W S
    float o[N8][4];
#pragma unroll
    for (int n = 0; n < N8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    Frag fp[2], fk[2][2];                           // P and K'^T (two blocks of S) of a 16-row step
    {
      uint32_t bh[2][N8 / 2][4], bl[2][N8 / 2][4];
#pragma unroll
      for (int n2 = 0; n2 < N8 / 2; ++n2) {
        ld_b(a_sh, 0, n2, bh[0][n2]);
        ld_b(a_sl, 0, n2, bl[0][n2]);
      }
#pragma unroll
      for (int kk = 0; kk < MAX_KD; ++kk) {
        if (kk >= kd) continue;
        if (kk + 2 < kd) {
          fq[(kk + 2) % 3] = load_frag(id.unit, lay.q + warp * kd + kk + 2, lane);
          if (DELTA) fw[(kk + 2) % 3] = load_frag(id.unit, lay.w + warp * kd + kk + 2, lane);
        }
        if (kk + 1 < kd)
#pragma unroll
          for (int n2 = 0; n2 < N8 / 2; ++n2) {
            ld_b(a_sh, kk + 1, n2, bh[(kk + 1) & 1][n2]);
            ld_b(a_sl, kk + 1, n2, bl[(kk + 1) & 1][n2]);
          }
        if (kk == kd - 1) {                         // what follows the barrier
          fp[0] = load_frag(id.unit, lay.p + warp * (warp + 1) / 2, lane);
          if (warp < kd) fk[0][0] = load_frag(id.unit, lay.k + warp * 4, lane);
          if (warp + 4 < kd) fk[0][1] = load_frag(id.unit, lay.k + (warp + 4) * 4, lane);
        }
        Frag& q = fq[kk % 3];
        Frag& w = fw[kk % 3];
        if (DELTA)
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            w.h[x] ^= 0x80008000u;
            w.l[x] ^= 0x80008000u;
          }
#pragma unroll
        for (int n = 0; n < N8; ++n) {
          const uint32_t *hh = bh[kk & 1][n / 2] + (n & 1) * 2, *ll = bl[kk & 1][n / 2] + (n & 1) * 2;
          mma3(o[n], q, hh[0], hh[1], ll[0], ll[1]);
          if (DELTA) mma3(u[n], w, hh[0], hh[1], ll[0], ll[1]);
        }
      }
    }
#pragma unroll
    for (int n = 0; n < N8; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int off = (i0 + half * 8) * PITCH + n * 8 + gc;
        uint32_t hi, lo;
        split_pack(u[n][half * 2], u[n][half * 2 + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(s_uh + off) = hi;
        if (DELTA) *reinterpret_cast<uint32_t*>(s_ul + off) = lo;  // a bf16 value has no second term
      }
    const float* dec = reinterpret_cast<const float*>(id.unit + lay.dec);
#pragma unroll
    for (int mi = 0; mi < 2; ++mi) {
      if (warp + mi * 4 >= kd) continue;
      const float d0 = __ldcg(dec + (warp + mi * 4) * 16 + gr), d1 = __ldcg(dec + (warp + mi * 4) * 16 + gr + 8);
#pragma unroll
      for (int n = 0; n < N8; ++n) {
        S[mi][n][0] *= d0;
        S[mi][n][1] *= d0;
        S[mi][n][2] *= d1;
        S[mi][n][3] *= d1;
      }
    }
    __syncthreads();
    const ChunkId now = id;
    // ---- O += P U, S = dec S + K'^T U
    {
      uint32_t bh[2][N8 / 2][4], bl[2][N8 / 2][4];
#pragma unroll
      for (int n2 = 0; n2 < N8 / 2; ++n2) {
        ld_b(a_uh, 0, n2, bh[0][n2]);
        if (DELTA) ld_b(a_ul, 0, n2, bl[0][n2]);
      }
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt < 3) {
          if (kt + 1 <= warp) fp[(kt + 1) & 1] = load_frag(now.unit, lay.p + warp * (warp + 1) / 2 + kt + 1, lane);
          if (warp < kd) fk[(kt + 1) & 1][0] = load_frag(now.unit, lay.k + warp * 4 + kt + 1, lane);
          if (warp + 4 < kd) fk[(kt + 1) & 1][1] = load_frag(now.unit, lay.k + (warp + 4) * 4 + kt + 1, lane);
#pragma unroll
          for (int n2 = 0; n2 < N8 / 2; ++n2) {
            ld_b(a_uh, kt + 1, n2, bh[(kt + 1) & 1][n2]);
            if (DELTA) ld_b(a_ul, kt + 1, n2, bl[(kt + 1) & 1][n2]);
          }
        } else if (c + 1 < n_chunks) {
          chunk_of(p, lay, c + 1, h, b, id);
          fetch(id);
        }
        auto add = [&](float (&acc)[4], const Frag& f, int n) {
          const uint32_t* hh = bh[kt & 1][n / 2] + (n & 1) * 2;
          if (DELTA) {
            const uint32_t* ll = bl[kt & 1][n / 2] + (n & 1) * 2;
            mma3(acc, f, hh[0], hh[1], ll[0], ll[1]);
          } else {
            mma_bf16(acc, f.l, hh[0], hh[1]);
            mma_bf16(acc, f.h, hh[0], hh[1]);
          }
        };
#pragma unroll
        for (int n = 0; n < N8; ++n) {
          if (kt <= warp) add(o[n], fp[kt & 1], n);
          if (warp < kd) add(S[0][n], fk[kt & 1][0], n);
          if (warp + 4 < kd) add(S[1][n], fk[kt & 1][1], n);
        }
      }
    }
#pragma unroll
    for (int n = 0; n < N8; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = i0 + half * 8, v = v0 + n * 8 + gc;
        if (i < now.n && v < p.V)
          *reinterpret_cast<float2*>(p.o_raw + ((long long)(now.row0 + i) * p.H + h) * p.V + v) =
              make_float2(o[n][half * 2], o[n][half * 2 + 1]);
        else if (MEM && i < now.n && v == p.V)
          p.den[(long long)(now.row0 + i) * p.H + h] = o[n][half * 2];
      }
    put_state();                                    // the products with the old state ended before the barrier above
    __syncthreads();
  }
  state_io(false);
}

template <int KIND>
static void launch_chunks(const StepParams& p, int max_len, cudaStream_t s) {
  constexpr bool DELTA = KIND == REC_DELTA;
  const ChunkLayout lay = chunk_layout(p.D, p.V, DELTA);
  const int chunks = (max_len + CK - 1) / CK, pitch = chunk_pitch(lay.kd);
  const dim3 grid(chunks, p.H, p.runs.B);
  if (DELTA) {
    const int smem = (CK * pitch + CK * (pitch > CA_THREADS / 2 ? pitch : CA_THREADS / 2) + CK * CK + 5 * CK) * 4;
    cudaFuncSetAttribute(delta_chunk_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    delta_chunk_prepare_kernel<<<grid, CA_THREADS, smem, s>>>(p);
  } else if (KIND == REC_MEMORY) {
    const int smem = (2 * CK * pitch + 2 * CK) * 4;
    cudaFuncSetAttribute(memory_chunk_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    memory_chunk_prepare_kernel<<<grid, CA_THREADS, smem, s>>>(p);
  } else {
    const int smem = (3 * CK * pitch + 4 * 16 * 18) * 4;
    cudaFuncSetAttribute(gla_chunk_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    gla_chunk_prepare_kernel<<<grid, CA_THREADS, smem, s>>>(p);
  }
  const int columns = p.V + (KIND == REC_MEMORY ? 1 : 0);
  auto scan = [&](auto kern, int vb) {
    const int smem = 2 * (lay.kd * 16 + CK) * (vb + 8) * 2;
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    kern<<<dim3((columns + vb - 1) / vb, p.H, p.runs.B), CB_THREADS, smem, s>>>(p);
  };
  // few (request, head) pairs: narrower column blocks for more CTAs
  if (p.runs.B * p.H * ((p.V + 31) / 32) >= 2 * 148) scan(chunk_scan_kernel<KIND, 32>, 32);
  else scan(chunk_scan_kernel<KIND, 16>, 16);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("chunked recurrence: ") + cudaGetErrorString(e));
}
void launch_gla_chunk(const StepParams& p, int max_len, cudaStream_t s) { launch_chunks<REC_GLA>(p, max_len, s); }
void launch_delta_chunk(const StepParams& p, int max_len, cudaStream_t s) { launch_chunks<REC_DELTA>(p, max_len, s); }
void launch_memory_chunk(const StepParams& p, int max_len, cudaStream_t s) { launch_chunks<REC_MEMORY>(p, max_len, s); }

}  // namespace fc
