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
