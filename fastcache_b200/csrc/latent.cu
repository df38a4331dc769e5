// Latent attention around the cache: norms of the latents, rotation of the shared key part and of the queries, store of
// the cache rows, gather of a request's rows for the expanded form, and the general (any size, fp32 or bf16) form of
// attention over paged rows that all heads share.
#include <algorithm>
#include <stdexcept>
#include <string>

#include "hybrid.cuh"
#include "launch.h"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int LS_THREADS = 256;

// column r of a rotated part whose first column is `col` of the projection; cs: cos | sin, rot_dims / 2 each
template <typename T>
__device__ __forceinline__ float turned_at(const LatentStore& p, long long t, int col, int r, const float* cs) {
  const float v = proj_at<T>(p.proj, t, col + r);
  if (r >= p.rot_dims) return v;
  const int half = p.rot_dims / 2;
  const bool first = p.half ? r < half : (r & 1) == 0;
  const int i = p.half ? (first ? r : r - half) : r >> 1, step = p.half ? half : 1;
  const float o = proj_at<T>(p.proj, t, col + r + (first ? step : -step));
  return first ? v * cs[i] - o * cs[half + i] : v * cs[i] + o * cs[half + i];
}
// cache row of token t: normed latent | rotated shared key part; by the whole CTA
template <typename T, int THREADS>
__device__ __forceinline__ void store_latent_row(const LatentStore& p, long long t, const float* cs, float* red) {
  const int slot = p.slots[t];
  if (slot < 0) return;
  if (slot >= p.num_rows) {
    if (threadIdx.x == 0) report(p.status, ST_BAD_INDEX);
    return;
  }
  T* row = reinterpret_cast<T*>(p.pool) + (long long)slot * p.row_width;
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.rank; c += THREADS) {
    const float v = proj_at<T>(p.proj, t, p.off_kv + c);
    ss += v * v;
  }
  const float inv = rsqrtf(cta_sum<THREADS>(ss, red) / float(p.rank) + p.eps);
  for (int c = threadIdx.x; c < p.rank; c += THREADS)
    row[c] = Elem<T>::put(proj_at<T>(p.proj, t, p.off_kv + c) * inv * p.norm_w[c]);
  for (int r = threadIdx.x; r < p.R; r += THREADS)
    row[p.rank + r] = Elem<T>::put(turned_at<T>(p, t, p.off_kv + p.rank, r, cs));
}

template <typename T>
__global__ void __launch_bounds__(LS_THREADS)
latent_store_kernel(const LatentStore p) {
  __shared__ float red[LS_THREADS / 32];
  extern __shared__ float cs[];                   // cos | sin of this token, rot_dims / 2 each
  const int half = p.rot_dims / 2;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const double pos = double(p.positions[t]);
  for (int i = threadIdx.x; i < half; i += LS_THREADS) turn_angle(pos, p.freq[i], cs[i], cs[half + i]);
  __syncthreads();
  const int part = blockIdx.y, parts = gridDim.y;
  // queries: every (head, column) of this part
  const int Q = p.D + p.R;
  T* q_abs = reinterpret_cast<T*>(p.q_abs);
  T* q = reinterpret_cast<T*>(p.q);
  const int qw = q_abs != nullptr ? p.D : Q;
  for (int idx = part * LS_THREADS + threadIdx.x; idx < p.H * Q; idx += parts * LS_THREADS) {
    const int h = idx / Q, c = idx - h * Q;
    const int r = c - p.D;
    const float v = r < 0 ? proj_at<T>(p.proj, t, p.off_q + idx) : turned_at<T>(p, t, p.off_q + idx - r, r, cs);
    if (r < 0 || q_abs == nullptr) q[(t * p.H + h) * qw + c] = Elem<T>::put(v);
    else q_abs[(t * p.H + h) * (p.rank + p.R) + p.rank + r] = Elem<T>::put(v);
  }
  if (p.gate != nullptr) {
    T* gate = reinterpret_cast<T*>(p.gate);
    for (int c = part * LS_THREADS + threadIdx.x; c < p.H * p.V; c += parts * LS_THREADS)
      gate[t * p.H * p.V + c] = Elem<T>::put(proj_at<T>(p.proj, t, p.off_g + c));
  }
  if (p.off_kv < 0 || part != 0) return;
  store_latent_row<T, LS_THREADS>(p, t, cs, red);
}

// The queries alone, four columns per access (sizes and offsets multiples of 4; where halves turn, half a rotated part as well)
template <typename T>
__global__ void __launch_bounds__(LS_THREADS)
latent_queries_kernel(const LatentStore p) {
  extern __shared__ float cs[];
  const int half = p.rot_dims / 2, Q = p.D + p.R, n = p.H * Q;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const int idx = (blockIdx.y * LS_THREADS + threadIdx.x) * 4, h = idx / Q, c = idx - h * Q, r = c - p.D;
  float4 v, o;
  const bool on = idx < n, turn = on && r >= 0 && r < p.rot_dims;
  if (on) v = proj_at4<T>(p.proj, t, p.off_q + idx);
  if (turn && p.half) o = proj_at4<T>(p.proj, t, p.off_q + idx + (r < half ? half : -half));
  const double pos = double(p.positions[t]);
  for (int i = threadIdx.x; i < half; i += LS_THREADS) turn_angle(pos, p.freq[i], cs[i], cs[half + i]);
  __syncthreads();
  if (!on) return;
  if (turn && p.half) {
    const int i = r < half ? r : r - half;
    const float f = r < half ? -1.f : 1.f;
    const float4 a = *reinterpret_cast<const float4*>(cs + i), b = *reinterpret_cast<const float4*>(cs + half + i);
    v = make_float4(v.x * a.x + f * o.x * b.x, v.y * a.y + f * o.y * b.y, v.z * a.z + f * o.z * b.z, v.w * a.w + f * o.w * b.w);
  } else if (turn) {
    const float2 a = *reinterpret_cast<const float2*>(cs + r / 2), b = *reinterpret_cast<const float2*>(cs + half + r / 2);
    v = make_float4(v.x * a.x - v.y * b.x, v.y * a.x + v.x * b.x, v.z * a.y - v.w * b.y, v.w * a.y + v.z * b.y);
  }
  T* q = reinterpret_cast<T*>(p.q);
  if (p.q_abs == nullptr) store4(q + t * n + idx, v.x, v.y, v.z, v.w);
  else if (r < 0) store4(q + (t * p.H + h) * p.D + c, v.x, v.y, v.z, v.w);
  else store4(reinterpret_cast<T*>(p.q_abs) + (t * p.H + h) * (p.rank + p.R) + p.rank + r, v.x, v.y, v.z, v.w);
}
static bool latent_queries_supported(const LatentStore& p) {
  return p.off_kv < 0 && p.gate == nullptr && p.D % 4 == 0 && p.R % 4 == 0 && p.rank % 4 == 0 && p.off_q % 4 == 0 && p.rot_dims % 4 == 0 &&
         (!p.half || p.rot_dims % 8 == 0);
}

// Normed query latent, cache row and head gates of a token (the queries are made from the query latent afterwards).  VEC: four
// columns per access, everything read ahead of one barrier
constexpr int LI_Q = 4, LI_KV = 1;                       // four-column pieces per thread: q_rank up to 4096, rank up to 1024
template <typename T, bool VEC>
__global__ void __launch_bounds__(LS_THREADS)
latent_inputs_kernel(const LatentStore p) {
  __shared__ float2 red2[LS_THREADS / 32];
  __shared__ float red[LS_THREADS / 32];
  extern __shared__ float cs[];
  const int half = p.rot_dims / 2, tid = threadIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  T* cq = reinterpret_cast<T*>(p.cq) + t * p.ld_cq;
  if constexpr (!VEC) {
    const double pos = double(p.positions[t]);
    for (int i = tid; i < half; i += LS_THREADS) turn_angle(pos, p.freq[i], cs[i], cs[half + i]);
    float ss = 0.f;
    for (int c = tid; c < p.q_rank; c += LS_THREADS) {
      const float v = proj_at<T>(p.proj, t, p.off_dq + c);
      ss += v * v;
    }
    const float inv = rsqrtf(cta_sum<LS_THREADS>(ss, red) / float(p.q_rank) + p.eps);      // also makes cs visible
    for (int c = tid; c < p.ld_cq; c += LS_THREADS)
      cq[c] = Elem<T>::put(c < p.q_rank ? proj_at<T>(p.proj, t, p.off_dq + c) * inv * p.q_norm_w[c] : 0.f);
    if (p.head_gate != nullptr)
      for (int h = tid; h < p.H; h += LS_THREADS) p.head_gate[t * p.H + h] = sigmoid_f(proj_at<T>(p.proj, t, p.off_g + h));
    if (p.off_kv >= 0) store_latent_row<T, LS_THREADS>(p, t, cs, red);
  } else {
    float4 q[LI_Q], kv[LI_KV];
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < LI_Q; ++i) {
      const int c = (tid + i * LS_THREADS) * 4;
      if (c < p.q_rank) q[i] = proj_at4<T>(p.proj, t, p.off_dq + c);
    }
#pragma unroll
    for (int i = 0; i < LI_KV; ++i) {
      const int c = (tid + i * LS_THREADS) * 4;
      if (c < p.rank) kv[i] = proj_at4<T>(p.proj, t, p.off_kv + c);
    }
    // rotated part and gates by the last threads
    const int lt = LS_THREADS - 1 - tid, slot = p.slots[t];
    const bool turn = lt < half;
    float u = 0.f, v = 0.f, c = 1.f, s = 0.f;
    const int cu = p.half ? lt : 2 * lt, cv = p.half ? half + lt : 2 * lt + 1, rot = p.off_kv + p.rank;
    if (turn) {
      u = proj_at<T>(p.proj, t, rot + cu);
      v = proj_at<T>(p.proj, t, rot + cv);
      turn_angle(double(p.positions[t]), p.freq[lt], c, s);
    }
    if (p.head_gate != nullptr)
      for (int h = tid; h < p.H; h += LS_THREADS) p.head_gate[t * p.H + h] = sigmoid_f(proj_at<T>(p.proj, t, p.off_g + h));
#pragma unroll
    for (int i = 0; i < LI_Q; ++i)
      if ((tid + i * LS_THREADS) * 4 < p.q_rank) sq += q[i].x * q[i].x + q[i].y * q[i].y + q[i].z * q[i].z + q[i].w * q[i].w;
#pragma unroll
    for (int i = 0; i < LI_KV; ++i)
      if ((tid + i * LS_THREADS) * 4 < p.rank) sk += kv[i].x * kv[i].x + kv[i].y * kv[i].y + kv[i].z * kv[i].z + kv[i].w * kv[i].w;
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((tid & 31) == 0) red2[tid >> 5] = make_float2(sq, sk);
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < LS_THREADS / 32; ++i) {
      sq += red2[i].x;
      sk += red2[i].y;
    }
    const float iq = rsqrtf(sq / float(p.q_rank) + p.eps), ik = rsqrtf(sk / float(p.rank) + p.eps);
    auto put = [&](T* dst, const float4& x, const float* w, float inv) {
      const float4 g = *reinterpret_cast<const float4*>(w);
      store4(dst, x.x * inv * g.x, x.y * inv * g.y, x.z * inv * g.z, x.w * inv * g.w);
    };
#pragma unroll
    for (int i = 0; i < LI_Q; ++i) {
      const int at = (tid + i * LS_THREADS) * 4;
      if (at < p.q_rank) put(cq + at, q[i], p.q_norm_w + at, iq);
    }
    for (int at = p.q_rank + tid; at < p.ld_cq; at += LS_THREADS) cq[at] = Elem<T>::put(0.f);
    if (slot < 0) return;
    if (slot >= p.num_rows) {
      if (tid == 0) report(p.status, ST_BAD_INDEX);
      return;
    }
    T* row = reinterpret_cast<T*>(p.pool) + (long long)slot * p.row_width;
#pragma unroll
    for (int i = 0; i < LI_KV; ++i) {
      const int at = (tid + i * LS_THREADS) * 4;
      if (at < p.rank) put(row + at, kv[i], p.norm_w + at, ik);
    }
    if (turn) {
      row[p.rank + cu] = Elem<T>::put(u * c - v * s);
      row[p.rank + cv] = Elem<T>::put(v * c + u * s);
    }
  }
}
// The same for many rows of a finished projection (bf16): one warp per token, everything in flight at once.  NQ: 16-byte pieces of
// the query latent per lane
constexpr int LW_WARPS = 8, LW_KV = 4;
template <int NQ>
__global__ void __launch_bounds__(LW_WARPS * 32)
latent_inputs_rows_kernel(const LatentStore p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long t = (long long)blockIdx.x * LW_WARPS + (threadIdx.x >> 5);
  if (t >= p.T) return;
  const bf16* row = reinterpret_cast<const bf16*>(p.proj.p) + t * p.proj.ld;
  uint4 q[NQ], kv[LW_KV];
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int c = (lane + i * 32) * 8;
    q[i] = c < p.q_rank ? __ldcg(reinterpret_cast<const uint4*>(row + p.off_dq + c)) : make_uint4(0, 0, 0, 0);
  }
#pragma unroll
  for (int i = 0; i < LW_KV; ++i) {
    const int c = (lane + i * 32) * 8;
    kv[i] = c < p.rank ? __ldcg(reinterpret_cast<const uint4*>(row + p.off_kv + c)) : make_uint4(0, 0, 0, 0);
  }
  const int slot = p.slots[t], half = p.rot_dims / 2, rot = p.off_kv + p.rank;
  const double pos = double(p.positions[t]);
  if (p.head_gate != nullptr)
    for (int h = lane; h < p.H; h += 32) p.head_gate[t * p.H + h] = sigmoid_f(Elem<bf16>::get(row[p.off_g + h]));
  auto squares = [](const uint4& u) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float a = __uint_as_float(w[e] << 16), b = __uint_as_float(w[e] & 0xffff0000u);
      s += a * a + b * b;
    }
    return s;
  };
  auto put = [](bf16* dst, const uint4& u, const float* g, float inv) {
    const float4 a = *reinterpret_cast<const float4*>(g), b = *reinterpret_cast<const float4*>(g + 4);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
    const float f[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
    uint32_t o[4];
#pragma unroll
    for (int e = 0; e < 4; ++e)
      o[e] = pack_bf16(__uint_as_float(w[e] << 16) * inv * f[2 * e], __uint_as_float(w[e] & 0xffff0000u) * inv * f[2 * e + 1]);
    *reinterpret_cast<uint4*>(dst) = make_uint4(o[0], o[1], o[2], o[3]);
  };
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < NQ; ++i) sq += squares(q[i]);
#pragma unroll
  for (int i = 0; i < LW_KV; ++i) sk += squares(kv[i]);
  const float iq = rsqrtf(warp_sum(sq) / float(p.q_rank) + p.eps), ik = rsqrtf(warp_sum(sk) / float(p.rank) + p.eps);
  bf16* cq = reinterpret_cast<bf16*>(p.cq) + t * p.ld_cq;    // ld_cq == q_rank: a multiple of 8
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int c = (lane + i * 32) * 8;
    if (c < p.q_rank) put(cq + c, q[i], p.q_norm_w + c, iq);
  }
  if (slot < 0) return;
  if (slot >= p.num_rows) {
    if (lane == 0) report(p.status, ST_BAD_INDEX);
    return;
  }
  bf16* dst = reinterpret_cast<bf16*>(p.pool) + (long long)slot * p.row_width;
#pragma unroll
  for (int i = 0; i < LW_KV; ++i) {
    const int c = (lane + i * 32) * 8;
    if (c < p.rank) put(dst + c, kv[i], p.norm_w + c, ik);
  }
  for (int i = lane; i < half; i += 32) {
    const int cu = p.half ? i : 2 * i, cv = p.half ? half + i : 2 * i + 1;
    const float u = Elem<bf16>::get(row[rot + cu]), v = Elem<bf16>::get(row[rot + cv]);
    float c, s;
    turn_angle(pos, p.freq[i], c, s);
    dst[p.rank + cu] = Elem<bf16>::put(u * c - v * s);
    dst[p.rank + cv] = Elem<bf16>::put(v * c + u * s);
  }
}
static bool latent_inputs_rows(const LatentStore& p) {
  return p.T >= 256 && p.proj.part == nullptr && p.off_kv >= 0 && p.q_rank % 8 == 0 && p.q_rank <= 12 * 256 && p.rank % 8 == 0 &&
         p.rank <= LW_KV * 256 && p.off_dq % 8 == 0 && p.off_kv % 8 == 0 && p.proj.ld % 8 == 0 && p.row_width % 8 == 0 && p.rot_dims == p.R;
}
static bool latent_inputs_vec(const LatentStore& p) {
  return p.off_kv >= 0 && p.q_rank % 4 == 0 && p.q_rank <= LS_THREADS * 4 * LI_Q && p.rank % 4 == 0 && p.rank <= LS_THREADS * 4 * LI_KV &&
         p.off_dq % 4 == 0 && p.off_kv % 4 == 0 && p.rot_dims == p.R && p.R <= 2 * LS_THREADS;
}

// The same for many rows of a finished projection whose queries are then read where they are: the rotated parts are
// rotated in place, nothing is copied.  Four columns per access (sizes and offsets multiples of 4); one warp per row for
// the cache row, the other warps rotate the heads.
constexpr int LR_WARPS = 4;
template <typename T>
__global__ void __launch_bounds__(LR_WARPS * 32)
latent_rotate_kernel(const LatentStore p) {
  extern __shared__ float cs[];
  const int half = p.rot_dims / 2, quads = half / 4;        // quads of pairs
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const int tid = threadIdx.x, lane = tid & 31;
  const double pos = double(p.positions[t]);
  for (int i = tid; i < half; i += LR_WARPS * 32) turn_angle(pos, p.freq[i], cs[i], cs[half + i]);
  __syncthreads();
  T* row = const_cast<T*>(reinterpret_cast<const T*>(p.proj.p)) + t * p.proj.ld;
  auto rotate = [&](const T* su, T* du, int i0) {            // quads at columns i0 and half + i0 of a rotated part
    ProjSrc s;
    s.p = su;
    if (!p.half) {                                           // columns 2 i0 .. 2 i0 + 7
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const float4 a = proj_at4<T>(s, 0, 2 * (i0 + e));
        const float2 c = *reinterpret_cast<const float2*>(cs + i0 + e), d = *reinterpret_cast<const float2*>(cs + half + i0 + e);
        store4(du + 2 * (i0 + e), a.x * c.x - a.y * d.x, a.y * c.x + a.x * d.x, a.z * c.y - a.w * d.y, a.w * c.y + a.z * d.y);
      }
      return;
    }
    const float4 u = proj_at4<T>(s, 0, i0), v = proj_at4<T>(s, 0, half + i0);
    const float4 c = *reinterpret_cast<const float4*>(cs + i0), d = *reinterpret_cast<const float4*>(cs + half + i0);
    store4(du + i0, u.x * c.x - v.x * d.x, u.y * c.y - v.y * d.y, u.z * c.z - v.z * d.z, u.w * c.w - v.w * d.w);
    store4(du + half + i0, v.x * c.x + u.x * d.x, v.y * c.y + u.y * d.y, v.z * c.z + u.z * d.z, v.w * c.w + u.w * d.w);
  };
  for (int i = tid; i < p.H * quads; i += LR_WARPS * 32) {
    const int h = i / quads;
    T* q = row + p.off_q + h * (p.D + p.R) + p.D;
    rotate(q, q, (i - h * quads) * 4);
  }
  if (p.off_kv < 0 || tid >= 32) return;
  const int slot = p.slots[t];
  if (slot < 0) return;
  if (slot >= p.num_rows) {
    if (lane == 0) report(p.status, ST_BAD_INDEX);
    return;
  }
  T* dst = reinterpret_cast<T*>(p.pool) + (long long)slot * p.row_width;
  ProjSrc s;
  s.p = row + p.off_kv;
  float ss = 0.f;
  for (int c = lane * 4; c < p.rank; c += 128) {
    const float4 v = proj_at4<T>(s, 0, c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float inv = rsqrtf(warp_sum(ss) / float(p.rank) + p.eps);
  for (int c = lane * 4; c < p.rank; c += 128) {
    const float4 v = proj_at4<T>(s, 0, c), w = *reinterpret_cast<const float4*>(p.norm_w + c);
    store4(dst + c, v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w);
  }
  for (int i = lane; i < quads; i += 32) rotate(row + p.off_kv + p.rank, dst + p.rank, i * 4);
}
bool latent_rotate_supported(const LatentStore& p) {
  return p.proj.splits <= 1 && p.rot_dims == p.R && p.R % 8 == 0 && p.D % 4 == 0 && p.rank % 4 == 0;
}

void launch_latent_inputs(const LatentStore& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  const size_t smem = size_t(std::max(2, p.rot_dims)) * 4;
  if (!f32 && latent_inputs_rows(p)) {
    auto go = [&](auto kern) { launch_pdl(PDL_ROPE, kern, dim3((p.T + LW_WARPS - 1) / LW_WARPS), dim3(LW_WARPS * 32), 0, s, p); };
    if (p.q_rank <= 4 * 256) go(latent_inputs_rows_kernel<4>);
    else if (p.q_rank <= 8 * 256) go(latent_inputs_rows_kernel<8>);
    else go(latent_inputs_rows_kernel<12>);
    const cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) throw std::runtime_error(std::string("latent inputs: ") + cudaGetErrorString(e));
    return;
  }
  auto go = [&](auto kern) { launch_pdl(PDL_ROPE, kern, dim3(p.T), dim3(LS_THREADS), smem, s, p); };
  const bool vec = latent_inputs_vec(p);
  if (f32) vec ? go(latent_inputs_kernel<float, true>) : go(latent_inputs_kernel<float, false>);
  else vec ? go(latent_inputs_kernel<bf16, true>) : go(latent_inputs_kernel<bf16, false>);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("latent inputs: ") + cudaGetErrorString(e));
}

void launch_latent_store(const LatentStore& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (p.q == nullptr) {                                      // in place
    if (!latent_rotate_supported(p)) throw std::runtime_error("latent store: queries cannot stay in place");
    const size_t smem = size_t(p.rot_dims) * 4;
    if (f32) launch_pdl(PDL_ROPE, latent_rotate_kernel<float>, dim3(p.T), dim3(LR_WARPS * 32), smem, s, p);
    else launch_pdl(PDL_ROPE, latent_rotate_kernel<bf16>, dim3(p.T), dim3(LR_WARPS * 32), smem, s, p);
    const cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) throw std::runtime_error(std::string("latent store: ") + cudaGetErrorString(e));
    return;
  }
  const int work = p.H * (p.D + p.R);
  if (latent_queries_supported(p)) {
    const dim3 grid(p.T, (work + LS_THREADS * 4 - 1) / (LS_THREADS * 4));
    const size_t smem = size_t(std::max(2, p.rot_dims)) * 4;
    if (f32) launch_pdl(PDL_ROPE, latent_queries_kernel<float>, grid, dim3(LS_THREADS), smem, s, p);
    else launch_pdl(PDL_ROPE, latent_queries_kernel<bf16>, grid, dim3(LS_THREADS), smem, s, p);
    const cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) throw std::runtime_error(std::string("latent store: ") + cudaGetErrorString(e));
    return;
  }
  const int parts = p.T >= 592 ? 1 : std::max(1, std::min(16, (work + LS_THREADS * 4 - 1) / (LS_THREADS * 4)));
  const dim3 grid(p.T, parts);
  const size_t smem = size_t(std::max(2, p.rot_dims)) * 4;
  if (f32) launch_pdl(PDL_ROPE, latent_store_kernel<float>, grid, dim3(LS_THREADS), smem, s, p);
  else launch_pdl(PDL_ROPE, latent_store_kernel<bf16>, grid, dim3(LS_THREADS), smem, s, p);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("latent store: ") + cudaGetErrorString(e));
}

// ------------------------------------------------------------------ gather
// the last cu_kv[b + 1] - cu_kv[b] of the ctx[b] rows of every request, one after another, 16 bytes per thread
template <int BYTES>
__global__ void __launch_bounds__(256)
gather_rows_kernel(const uint8_t* __restrict__ pool, const int* __restrict__ block_tables, const int* __restrict__ ctx,
                   const int* __restrict__ cu_kv, uint8_t* __restrict__ out, int chunks, int block_size,
                   int max_blocks, int num_blocks, uint32_t* status) {
  const int b = blockIdx.y;
  const int len = min(ctx[b], max_blocks * block_size), n = min(len, cu_kv[b + 1] - cu_kv[b]);
  const int per = 256 / chunks > 0 ? 256 / chunks : 1;
  const int row0 = blockIdx.x * per;
  for (int i = threadIdx.x; i < per * chunks; i += 256) {
    const int row = row0 + i / chunks, c = i % chunks;
    if (row >= n) return;
    const int at = len - n + row, blk = block_tables[(long long)b * max_blocks + at / block_size];
    if (blk < 0 || blk >= num_blocks) {
      report(status, ST_BAD_INDEX);
      continue;
    }
    const long long src = (long long)blk * block_size + at % block_size;
    reinterpret_cast<uint4*>(out)[((long long)cu_kv[b] + row) * chunks + c] =
        reinterpret_cast<const uint4*>(pool)[src * chunks + c];
  }
}

void launch_gather_rows(const void* pool, const int* block_tables, const int* ctx, const int* cu_kv, void* out,
                        int B, int max_ctx, int row_width, int block_size, int max_blocks, int num_blocks, bool f32,
                        uint32_t* status, cudaStream_t s) {
  if (B == 0 || max_ctx == 0) return;
  const int chunks = row_width * (f32 ? 4 : 2) / 16;
  const int per = std::max(1, 256 / chunks);
  gather_rows_kernel<16><<<dim3((max_ctx + per - 1) / per, B), 256, 0, s>>>(
      (const uint8_t*)pool, block_tables, ctx, cu_kv, (uint8_t*)out, chunks, block_size, max_blocks, num_blocks, status);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("gather rows: ") + cudaGetErrorString(e));
}

// ------------------------------------------------------------------ attention over shared rows, general form
constexpr int LA_THREADS = 128;
constexpr int LA_TILE = 64;
constexpr int LA_COLS = 8;           // value columns per thread: up to 1024 per head

template <typename T>
__global__ void __launch_bounds__(LA_THREADS)
row_attn_simt_kernel(const RowAttn p) {
  extern __shared__ float sq[];                    // K query values
  __shared__ float ss[LA_TILE];
  __shared__ const T* srow[LA_TILE];
  const int t = blockIdx.x, h = blockIdx.y;
  const int ctx = min(p.row_ctx[t], p.max_blocks * p.block_size);
  const int b = p.row_seq != nullptr ? p.row_seq[t] : t;
  const int first = p.window > 0 ? max(0, ctx - p.window) : 0, vc = p.v_col + h / (p.H / p.v_heads) * p.V;
  const T* q = reinterpret_cast<const T*>(p.q) + ((long long)t * p.H + h) * p.K;
  const T* pool = reinterpret_cast<const T*>(p.pool);
  const int* bt = p.block_tables + (long long)b * p.max_blocks;
  for (int c = threadIdx.x; c < p.K; c += LA_THREADS) sq[c] = ctx > 0 ? Elem<T>::get(q[c]) * p.scale : 0.f;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float acc[LA_COLS];
#pragma unroll
  for (int i = 0; i < LA_COLS; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int k0 = first; k0 < ctx; k0 += LA_TILE) {
    const int n = min(LA_TILE, ctx - k0);
    __syncthreads();
    if (threadIdx.x < n) {
      const int j = k0 + threadIdx.x;
      int blk = bt[j / p.block_size];
      if (blk < 0 || blk >= p.num_blocks) {
        report(p.status, ST_BAD_INDEX);
        blk = 0;
      }
      srow[threadIdx.x] = pool + ((long long)blk * p.block_size + j % p.block_size) * p.row_width;
    }
    __syncthreads();
    for (int j = warp; j < n; j += LA_THREADS / 32) {
      float d = 0.f;
      for (int c = lane; c < p.K; c += 32) d = fmaf(sq[c], Elem<T>::get(srow[j][c]), d);
      d = warp_sum(d);
      if (lane == 0) ss[j] = d;
    }
    __syncthreads();
    float mx = m;
    for (int j = 0; j < n; ++j) mx = fmaxf(mx, ss[j]);
    const float corr = expf(m - mx);
    m = mx;
    l *= corr;
#pragma unroll
    for (int i = 0; i < LA_COLS; ++i) acc[i] *= corr;
    for (int j = 0; j < n; ++j) {
      const float e = expf(ss[j] - mx);
      l += e;
#pragma unroll
      for (int i = 0; i < LA_COLS; ++i) {
        const int c = threadIdx.x + i * LA_THREADS;
        if (c < p.V) acc[i] = fmaf(e, Elem<T>::get(srow[j][vc + c]), acc[i]);
      }
    }
  }
  if (p.sink != nullptr && ctx > 0) l += expf(p.sink[h] - m);
  float inv = l > 0.f ? 1.f / l : 0.f;
  if (p.head_gate != nullptr) inv *= p.head_gate[(long long)t * p.H + h];
  T* o = reinterpret_cast<T*>(p.out) + t * p.ld_out + h * p.V;
#pragma unroll
  for (int i = 0; i < LA_COLS; ++i) {
    const int c = threadIdx.x + i * LA_THREADS;
    if (c < p.V) o[c] = Elem<T>::put(acc[i] * inv);
  }
}

void launch_row_attn_simt(const RowAttn& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (p.V > LA_THREADS * LA_COLS) throw std::runtime_error("attention over shared rows: values are limited to 1024 columns (kv_rank)");
  const dim3 grid(p.T, p.H);
  const size_t smem = size_t(p.K) * 4;
  auto go = [&](auto kern) {
    if (smem > 40 * 1024) {
      if (smem > 200 * 1024) throw std::runtime_error("attention over shared rows: scores are limited to 50000 columns");
      cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    }
    kern<<<grid, LA_THREADS, smem, s>>>(p);
  };
  if (f32) go(row_attn_simt_kernel<float>);
  else go(row_attn_simt_kernel<bf16>);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("attention over shared rows: ") + cudaGetErrorString(e));
}

}  // namespace fc
