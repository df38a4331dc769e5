// Attention over per-head K/V rows: bias, norm over the whole query and key projections, rotation, cache store (the values
// may be the raw keys), and the general form of attention with window, chunks, soft cap, sink and output gate (any head size,
// bf16 or fp32; the tensor-core forms are attn_prefill*.cu and attn_decode.cu with AttnOptions).
#include <algorithm>
#include <stdexcept>
#include <string>

#include "attn_options.cuh"
#include "hybrid.cuh"
#include "launch.h"

namespace fc {

using bf16 = __nv_bfloat16;

// One CTA per token.  The projections are staged in shared memory as fp32 while their squares are summed; VEC: four
// columns at a time (head sizes, half of the rotated dimensions where halves turn, pitch and offsets multiples of 4).
template <typename T, bool VEC, int WS_THREADS>
__global__ void __launch_bounds__(WS_THREADS)
window_store_kernel(const WindowStore p) {
  __shared__ float2 red[WS_THREADS / 32];
  extern __shared__ __align__(16) float sm[];
  const int nq = p.H * p.D, nk = p.G * p.D, half = p.rot_dims / 2;
  const T* bias = reinterpret_cast<const T*>(p.bias);
  float *s_q = sm, *s_k = sm + nq;
  float2* cs = reinterpret_cast<float2*>(sm + ((nq + nk + 3) / 4) * 4);      // (cos, sin) of every pair
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const int tid = threadIdx.x;
  T* out = reinterpret_cast<T*>(p.out);
  if (tid < p.pad_out) out[t * p.ld_out + p.H * p.V + tid] = Elem<T>::put(0.f);
  const double pos = double(p.positions[t]);
  float sq = 0.f, sk = 0.f;
  // columns of the projection with their bias
  auto col1 = [&](int c) {
    const float v = proj_at<T>(p.proj, t, c);
    return bias != nullptr ? v + Elem<T>::get(bias[c]) : v;
  };
  auto col4 = [&](int c) {
    float4 v = proj_at4<T>(p.proj, t, c);
    if (bias != nullptr) {
      v.x += Elem<T>::get(bias[c]);
      v.y += Elem<T>::get(bias[c + 1]);
      v.z += Elem<T>::get(bias[c + 2]);
      v.w += Elem<T>::get(bias[c + 3]);
    }
    return v;
  };
  const int ng = p.H * p.V;
  if (VEC) {
#pragma unroll 4
    for (int i = tid * 4; i < nq; i += WS_THREADS * 4) {
      const float4 v = col4(p.off_q + i);
      *reinterpret_cast<float4*>(s_q + i) = v;
      sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    for (int i = tid * 4; i < nk; i += WS_THREADS * 4) {
      const float4 v = col4(p.off_k + i);
      *reinterpret_cast<float4*>(s_k + i) = v;
      sk += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    if (p.gate != nullptr)
      for (int i = tid * 4; i < ng; i += WS_THREADS * 4) {
        const float4 v = col4(p.off_g + i);
        store4(reinterpret_cast<T*>(p.gate) + t * ng + i, v.x, v.y, v.z, v.w);
      }
  } else {
    for (int i = tid; i < nq; i += WS_THREADS) {
      const float v = col1(p.off_q + i);
      s_q[i] = v;
      sq += v * v;
    }
    if (p.gate != nullptr)
      for (int i = tid; i < ng; i += WS_THREADS) reinterpret_cast<T*>(p.gate)[t * ng + i] = Elem<T>::put(col1(p.off_g + i));
    for (int i = tid; i < nk; i += WS_THREADS) {
      const float v = col1(p.off_k + i);
      s_k[i] = v;
      sk += v * v;
    }
  }
  for (int i = tid; i < half; i += WS_THREADS) {
    float c, s;
    turn_angle(pos, p.freq[i], c, s);
    cs[i] = make_float2(c * p.rot_size, s * p.rot_size);
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((tid & 31) == 0) red[tid >> 5] = make_float2(sq, sk);
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < WS_THREADS / 32; ++i) {
    sq += red[i].x;
    sk += red[i].y;
  }
  const float iq = rsqrtf(sq / float(nq) + p.eps), ik = rsqrtf(sk / float(nk) + p.eps);
  // column c of a head whose first element is x[0] and norm weight w[0]
  auto turned = [&](const float* x, const float* w, int c, float inv) {
    const float v = x[c] * inv * w[c];
    if (c >= p.rot_dims) return v;
    if (p.half) {
      const bool lo = c < half;
      const int d = lo ? c + half : c - half;
      const float2 a = cs[lo ? c : d];
      const float o = x[d] * inv * w[d];
      return lo ? v * a.x - o * a.y : v * a.x + o * a.y;
    }
    const float2 a = cs[c >> 1];
    const float o = x[c ^ 1] * inv * w[c ^ 1];
    return (c & 1) ? v * a.x + o * a.y : v * a.x - o * a.y;
  };
  auto normed = [&](const float* x, const float* w, int c, float inv) {
    const float4 v = *reinterpret_cast<const float4*>(x + c), g = *reinterpret_cast<const float4*>(w + c);
    return make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w);
  };
  auto four = [&](const float* x, const float* w, int c, float inv) {
    float4 y = normed(x, w, c, inv);
    if (p.half) {
      if (c >= p.rot_dims) return y;
      const bool lo = c < half;
      const int d = lo ? c + half : c - half;
      const float4 o = normed(x, w, d, inv);
      const float2* a = cs + (lo ? c : d);
      const float f = lo ? -1.f : 1.f;
      return make_float4(y.x * a[0].x + f * o.x * a[0].y, y.y * a[1].x + f * o.y * a[1].y, y.z * a[2].x + f * o.z * a[2].y,
                         y.w * a[3].x + f * o.w * a[3].y);
    }
    if (c < p.rot_dims) {
      const float2 a = cs[c >> 1];
      y = make_float4(y.x * a.x - y.y * a.y, y.y * a.x + y.x * a.y, y.z, y.w);
    }
    if (c + 2 < p.rot_dims) {
      const float2 a = cs[(c >> 1) + 1];
      y = make_float4(y.x, y.y, y.z * a.x - y.w * a.y, y.w * a.x + y.z * a.y);
    }
    return y;
  };
  T* q = reinterpret_cast<T*>(p.q) + t * p.H * p.pitch;
  constexpr int STEP = VEC ? 4 : 1;
  for (int i = tid * STEP; i < p.H * p.pitch; i += WS_THREADS * STEP) {
    const int h = i / p.pitch, c = i - h * p.pitch;
    if (VEC) {
      const float4 y = c < p.D ? four(s_q + h * p.D, p.q_norm + h * p.D, c, iq) : make_float4(0.f, 0.f, 0.f, 0.f);
      store4(q + i, y.x, y.y, y.z, y.w);
    } else {
      q[i] = Elem<T>::put(c < p.D ? turned(s_q + h * p.D, p.q_norm + h * p.D, c, iq) : 0.f);
    }
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  if (slot >= p.num_rows) {
    if (tid == 0) report(p.status, ST_BAD_INDEX);
    return;
  }
  const int blk = slot / p.block_size, off = slot - blk * p.block_size;
  for (int i = tid * STEP; i < p.G * p.pitch; i += WS_THREADS * STEP) {
    const int g = i / p.pitch, c = i - g * p.pitch;
    const long long dst = (((long long)blk * p.G + g) * p.block_size + off) * p.pitch + c;
    T *k = reinterpret_cast<T*>(p.k_rows) + dst, *v = reinterpret_cast<T*>(p.v_rows) + dst;
    const float* x = s_k + g * p.D;
    if (VEC) {
      const float4 y = c < p.D ? four(x, p.k_norm + g * p.D, c, ik) : make_float4(0.f, 0.f, 0.f, 0.f);
      store4(k, y.x, y.y, y.z, y.w);
      float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < p.V) r = p.off_v < 0 ? *reinterpret_cast<const float4*>(x + c) : col4(p.off_v + g * p.V + c);
      store4(v, r.x, r.y, r.z, r.w);
    } else {
      *k = Elem<T>::put(c < p.D ? turned(x, p.k_norm + g * p.D, c, ik) : 0.f);
      *v = Elem<T>::put(c >= p.V ? 0.f : p.off_v < 0 ? x[c] : col1(p.off_v + g * p.V + c));
    }
  }
}

// Many rows of heads that fill the pages' rows (bf16, finished projections).  A thread owns 16-byte pieces of the query and one
// of the key or the value of several tokens: the next token is requested ahead, the last threads make its angles meanwhile, and
// halves that turn together are exchanged within the warp.
constexpr int WR_MAX_HALF = 128;
__device__ __forceinline__ void unpack8(const uint4& u, float (&v)[8]) {
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    v[2 * i] = __uint_as_float(w[i] << 16);
    v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
__device__ __forceinline__ void add_bias8(float (&v)[8], const uint4& b) {
  float f[8];
  unpack8(b, f);
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] += f[e];
}
template <int THREADS, int NQ>
__global__ void __launch_bounds__(THREADS, NQ == 1 ? 1024 / THREADS : 1)
window_store_rows_kernel(const WindowStore p, int tokens) {
  __shared__ float2 red[2][THREADS / 32];
  __shared__ __align__(16) float2 cs[2][WR_MAX_HALF];
  const int tid = threadIdx.x, nq = p.H * p.D, nk = p.G * p.D, half = p.rot_dims / 2;
  const bool is_k = tid < nk / 8, is_v = !is_k && tid < nk / 4;
  const int at8 = (is_k ? tid : tid - nk / 8) * 8;           // first element of the key or value piece in its row
  const bf16 *src = reinterpret_cast<const bf16*>(p.proj.p), *bias = reinterpret_cast<const bf16*>(p.bias);
  const int kv_col = (is_k || p.off_v < 0 ? p.off_k : p.off_v) + at8;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  auto piece = [&](const bf16* row, int col) { return __ldcg(reinterpret_cast<const uint4*>(row + col)); };
  uint4 bq[NQ], bkv = zero;
#pragma unroll
  for (int j = 0; j < NQ; ++j) {
    const int i = (tid + j * THREADS) * 8;
    bq[j] = bias != nullptr && i < nq ? *reinterpret_cast<const uint4*>(bias + p.off_q + i) : zero;
  }
  if ((is_k || is_v) && bias != nullptr) bkv = *reinterpret_cast<const uint4*>(bias + kv_col);
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * tokens, t1 = min(p.T, t0 + tokens);
  if (t0 >= t1) return;
  uint4 q4[NQ], kv4 = zero;
#pragma unroll
  for (int j = 0; j < NQ; ++j) q4[j] = zero;
  int slot = 0;
  auto request = [&](int t) {
    const bf16* row = src + t * p.proj.ld;
#pragma unroll
    for (int j = 0; j < NQ; ++j)
      if ((tid + j * THREADS) * 8 < nq) q4[j] = piece(row, p.off_q + (tid + j * THREADS) * 8);
    if (is_k || is_v) kv4 = piece(row, kv_col);
    slot = p.slots[t];
  };
  request(t0);
  const int turn_i = THREADS - 1 - tid;                      // this thread's angle
  // halves that turn together read 16 bytes per pair of angles: the same pair of neighbouring pieces lies side by side
  const int turn_at = p.half ? (((turn_i & 7) >> 1) * (half >> 3) + (turn_i >> 3)) * 2 + (turn_i & 1) : turn_i;
  const double freq = turn_i < half ? p.freq[turn_i] : 0.0;
  auto angles = [&](int t) {
    if (turn_i >= half) return;
    float c, s;
    turn_angle(double(p.positions[t]), freq, c, s);
    cs[t & 1][turn_at] = make_float2(c * p.rot_size, s * p.rot_size);
  };
  angles(t0);
  // norm weight and rotation of a piece whose first column of the head is c; every lane of the warp takes part
  auto finish = [&](float (&y)[8], const float* w, float inv, int c, const float2* a, bool on) {
    if (on) {
      const float4 w0 = *reinterpret_cast<const float4*>(w), w1 = *reinterpret_cast<const float4*>(w + 4);
      const float f[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] *= inv * f[e];
    }
    if (half == 0) return;
    if (p.half) {
      const bool lo = c < half;
      const float f = lo ? -1.f : 1.f;
      const float4* g = reinterpret_cast<const float4*>(a) + ((c < p.rot_dims ? (lo ? c : c - half) : 0) >> 3);
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        const float o0 = __shfl_xor_sync(0xffffffffu, y[e], half >> 3), o1 = __shfl_xor_sync(0xffffffffu, y[e + 1], half >> 3);
        if (c < p.rot_dims) {
          const float4 gg = g[(e >> 1) * (half >> 3)];
          y[e] = y[e] * gg.x + f * o0 * gg.y;
          y[e + 1] = y[e + 1] * gg.z + f * o1 * gg.w;
        }
      }
    } else {
#pragma unroll
      for (int e = 0; e < 8; e += 2)
        if (c + e < p.rot_dims) {
          const float2 g = a[(c + e) >> 1];
          const float u = y[e], v = y[e + 1];
          y[e] = u * g.x - v * g.y;
          y[e + 1] = v * g.x + u * g.y;
        }
    }
  };
  for (int t = t0; t < t1; ++t) {
    const int par = t & 1, at = slot;
    float x[NQ][8], kv[8], sq = 0.f, sk = 0.f;
#pragma unroll
    for (int j = 0; j < NQ; ++j) {                           // pieces past the row are zero
      unpack8(q4[j], x[j]);
      add_bias8(x[j], bq[j]);
#pragma unroll
      for (int e = 0; e < 8; ++e) sq += x[j][e] * x[j][e];
    }
    unpack8(kv4, kv);
    add_bias8(kv, bkv);
    if (is_k)
#pragma unroll
      for (int e = 0; e < 8; ++e) sk += kv[e] * kv[e];
    if (t + 1 < t1) request(t + 1);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((tid & 31) == 0) red[par][tid >> 5] = make_float2(sq, sk);
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) {
      sq += red[par][i].x;
      sk += red[par][i].y;
    }
    const float iq = rsqrtf(sq / float(nq) + p.eps), ik = rsqrtf(sk / float(nk) + p.eps);
    const float2* turns = cs[par];
    if (t + 1 < t1) angles(t + 1);                           // of the buffer that was read before this token's barrier
    bf16* q = reinterpret_cast<bf16*>(p.q) + (long long)t * nq;
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
      const int i = (tid + j * THREADS) * 8;
      finish(x[j], p.q_norm + i, iq, i & (p.D - 1), turns, i < nq);
      if (i < nq) store8(q + i, x[j]);
    }
    if (tid < (nk / 8 + 31) / 32 * 32) {                     // whole warps; the value pieces among them stay as they are
      float y[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = kv[e];
      finish(y, p.k_norm + at8, ik, at8 & (p.D - 1), turns, is_k);
      if (is_k)
#pragma unroll
        for (int e = 0; e < 8; ++e) kv[e] = y[e];
    }
    if (at < 0 || !(is_k || is_v)) continue;
    if (at >= p.num_rows) {
      if (tid == 0) report(p.status, ST_BAD_INDEX);
      continue;
    }
    const int blk = at / p.block_size, off = at - blk * p.block_size;
    store8(reinterpret_cast<bf16*>(is_k ? p.k_rows : p.v_rows) +
               (((long long)blk * p.G + at8 / p.D) * p.block_size + off) * p.D + (at8 & (p.D - 1)), kv);
  }
}
static bool window_store_rows_supported(const WindowStore& p) {
  const int half = p.rot_dims / 2, shift = half / 8;
  const bool turn = half == 0 || (p.half ? half % 8 == 0 && shift <= 16 && (shift & (shift - 1)) == 0 && p.D % p.rot_dims == 0
                                         : half <= WR_MAX_HALF);
  return p.T >= 256 && p.proj.part == nullptr && p.gate == nullptr && (p.D == 64 || p.D == 128) && p.D == p.V && p.D == p.pitch && turn &&
         p.H * p.D <= 8192 && 2 * p.G * p.D <= (p.H * p.D <= 2048 ? 2048 : 4096) && p.proj.ld % 8 == 0 && p.off_q % 8 == 0 && p.off_k % 8 == 0 &&
         (p.off_v < 0 || p.off_v % 8 == 0) && p.pad_out == 0;
}
static void launch_window_store_rows(const WindowStore& p, cudaStream_t s) {
  auto go = [&](auto kern, int threads) {                    // two CTAs of 512 threads, four of 256 per SM
    const int ctas = 148 * 1024 / threads, tokens = std::max(4, (p.T + ctas - 1) / ctas);
    launch_pdl(PDL_ROPE, kern, dim3((p.T + tokens - 1) / tokens), dim3(threads), 0, s, p, tokens);
  };
  if (p.H * p.D <= 2048) go(window_store_rows_kernel<256, 1>, 256);
  else if (p.H * p.D <= 4096) go(window_store_rows_kernel<512, 1>, 512);
  else go(window_store_rows_kernel<512, 2>, 512);
}

// General form: one warp per (row, head).  A lane scores one of 32 keys, then the lanes share the value columns.
constexpr int WA_WARPS = 4;
template <typename T, int NACC>
__global__ void __launch_bounds__(WA_WARPS * 32)
window_attn_kernel(const WindowAttn p) {
  extern __shared__ __align__(16) float s_q_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y * WA_WARPS + warp;
  const long long t = blockIdx.x;
  if (h >= p.H) return;
  float* s_q = s_q_all + warp * p.D;
  const T* q = reinterpret_cast<const T*>(p.q) + (t * p.H + h) * p.pitch;
  for (int c = lane; c < p.D; c += 32) s_q[c] = Elem<T>::get(q[c]);
  __syncwarp();
  const int b = p.row_seq != nullptr ? p.row_seq[t] : int(t), ctx = p.row_ctx[t], g = h / (p.H / p.G);
  const int* bt = p.block_tables + (long long)b * p.max_blocks;
  AttnOptions seen;
  seen.window = p.window;
  seen.chunk = p.chunk;
  const int first = attn_first(seen, max(ctx - 1, 0));
  const T *kr = reinterpret_cast<const T*>(p.k_rows), *vr = reinterpret_cast<const T*>(p.v_rows);
  float acc[NACC];
#pragma unroll
  for (int i = 0; i < NACC; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int j0 = first; j0 < ctx; j0 += 32) {
    const int j = j0 + lane;
    long long row = -1;
    float s = -INFINITY;
    if (j < ctx) {
      const int at = j / p.block_size, blk = at < p.max_blocks ? bt[at] : -1;
      if (blk < 0 || blk >= p.num_blocks) {
        report(p.status, ST_BAD_INDEX);
      } else {
        row = (((long long)blk * p.G + g) * p.block_size + (j - at * p.block_size)) * p.pitch;
        s = 0.f;
        for (int c = 0; c < p.D; ++c) s = fmaf(s_q[c], Elem<T>::get(kr[row + c]), s);
        s *= p.scale;
        if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      }
    }
    __syncwarp();
    const float nm = fmaxf(m, warp_max(s));
    if (nm == -INFINITY) continue;
    const float f = m == -INFINITY ? 0.f : expf(m - nm), e = s == -INFINITY ? 0.f : expf(s - nm);
    m = nm;
    l = l * f + warp_sum(e);
#pragma unroll
    for (int i = 0; i < NACC; ++i) acc[i] *= f;
    for (int x = 0; x < min(32, ctx - j0); ++x) {
      const float pe = __shfl_sync(0xffffffffu, e, x);
      const long long pr = __shfl_sync(0xffffffffu, row, x);
      if (pr < 0) continue;
#pragma unroll
      for (int i = 0; i < NACC; ++i)
        if (lane + i * 32 < p.V) acc[i] = fmaf(pe, Elem<T>::get(vr[pr + lane + i * 32]), acc[i]);
    }
  }
  if (p.sink != nullptr && m != -INFINITY) l += expf(p.sink[h] - m);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T* out = reinterpret_cast<T*>(p.out) + t * p.ld_out + h * p.V;
#pragma unroll
  for (int i = 0; i < NACC; ++i) {
    const int c = lane + i * 32;
    if (c >= p.V) continue;
    const float gate = p.off_g >= 0 ? sigmoid_t<T>(proj_at<T>(p.gate, t, p.off_g + h * p.V + c)) : 1.f;
    out[c] = Elem<T>::put(acc[i] * inv * gate);
  }
}

// ================================================================= launchers
static void check_launch(const char* what) {
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string(what) + ": " + cudaGetErrorString(e));
}

template <typename T>
static void window_store_t(const WindowStore& p, cudaStream_t s) {
  const int n = (p.H + p.G) * p.D;
  const size_t smem = size_t((n + 3) / 4 * 4 + p.rot_dims) * 4;
  if (smem > 200 * 1024) throw std::runtime_error("windowed attention: query and key projections are limited to 50000 columns");
  const bool vec = p.D % 4 == 0 && p.V % 4 == 0 && p.pitch % 4 == 0 && p.off_q % 4 == 0 && p.off_k % 4 == 0 && p.off_g % 4 == 0 &&
                   (p.off_v < 0 || p.off_v % 4 == 0) && (!p.half || p.rot_dims % 8 == 0);
  auto go = [&](auto kern, int threads) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    launch_pdl(PDL_ROPE, kern, dim3(p.T), dim3(threads), smem, s, p);
  };
  if (vec && p.T <= 148) go(window_store_kernel<T, true, 1024>, 1024);      // one row per SM at most
  else if (vec) go(window_store_kernel<T, true, 256>, 256);
  else go(window_store_kernel<T, false, 256>, 256);
}
void launch_window_store(const WindowStore& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (f32) window_store_t<float>(p, s);
  else if (window_store_rows_supported(p)) launch_window_store_rows(p, s);
  else window_store_t<bf16>(p, s);
  check_launch("norm, rotation and store of windowed attention");
}

void launch_window_attn(const WindowAttn& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (p.D > 512 || p.V > 512) throw std::runtime_error("windowed attention: heads are limited to 512 columns");
  const dim3 grid(p.T, (p.H + WA_WARPS - 1) / WA_WARPS);
  const size_t smem = size_t(WA_WARPS) * p.D * 4;
  auto go = [&](auto kern) { kern<<<grid, WA_WARPS * 32, smem, s>>>(p); };
  if (f32) {
    if (p.V <= 128) go(window_attn_kernel<float, 4>);
    else go(window_attn_kernel<float, 16>);
  } else {
    if (p.V <= 128) go(window_attn_kernel<bf16, 4>);
    else go(window_attn_kernel<bf16, 16>);
  }
  check_launch("windowed attention");
}

}  // namespace fc
