// fp32 residual stream: embedding with a scale, norm of a sublayer's output + add, add + norm for the next sublayer, final
// norm, and the gates of feed-forwards.  Readers of a projection take split-K partial sums as they are.
#include <algorithm>
#include <stdexcept>
#include <string>

#include "hybrid.cuh"
#include "launch.h"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int RS_THREADS = 256;
constexpr int RS_CHUNKS = 8;        // 4-column chunks per thread: rows up to 8192 columns

template <typename T>
__global__ void __launch_bounds__(RS_THREADS)
embed_scaled_kernel(const long long* __restrict__ ids, const T* __restrict__ weight, float* __restrict__ x,
                    T* __restrict__ h, int W, int Wp, long long V, float scale, uint32_t* status) {
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  long long id = ids[row];
  const bool ok = id >= 0 && id < V;
  if (!ok) {
    if (threadIdx.x == 0) report(status, ST_BAD_INDEX);
    id = 0;
  }
  for (int c = threadIdx.x; c < Wp; c += RS_THREADS) {
    const float v = (c < W && ok) ? Elem<T>::get(weight[id * Wp + c]) * scale : 0.f;
    if (c < W) x[row * W + c] = v;
    h[row * Wp + c] = Elem<T>::put(v);
  }
}

// x += rms(f (y + bias) + mixed expert rows) * w;  h = x in the model's type, zero-padded from W to Wp columns.  NC: 4-column
// chunks per thread.  What does not depend on the norm is requested first
constexpr int PN_THREADS = 512, PN_TOP = 4;
template <typename T, bool VEC, int NC>
__global__ void __launch_bounds__(PN_THREADS)
post_norm_add_kernel(const PostNormAdd p) {
  __shared__ float red[PN_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  const int W = p.W;
  const T* bias = reinterpret_cast<const T*>(p.bias);
  float* x = p.x + row * W;
  T* h = reinterpret_cast<T*>(p.h) + row * p.Wp;
  auto col_of = [&](int c) { return (int(threadIdx.x) + c * PN_THREADS) * 4; };
  int r[PN_TOP];
  float f[PN_TOP];
#pragma unroll
  for (int j = 0; j < PN_TOP; ++j) {
    r[j] = j < p.top ? p.row_of[row * p.top + j] : -1;
    f[j] = j >= p.top ? 0.f : p.mix != nullptr ? p.mix[row * p.top + j] : 1.f / float(p.top);
  }
  const float fy = p.y_factor != nullptr ? p.y_factor[row] : 1.f;
  float4 xv[NC], v[NC];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    v[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (col >= W) continue;
    if (VEC) xv[c] = __ldcg(reinterpret_cast<const float4*>(x + col));
    if (p.has_y) v[c] = proj_at4<T>(p.y, row, col);      // the pad columns of a projection exist and are zero
  }
  auto add = [&](int rj, float fj) {
    if (rj < 0) return;
    float4 e[NC];
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (col_of(c) < W) e[c] = proj_at4<T>(p.experts, rj, col_of(c));
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (col_of(c) < W) {
        v[c].x = fmaf(e[c].x, fj, v[c].x);
        v[c].y = fmaf(e[c].y, fj, v[c].y);
        v[c].z = fmaf(e[c].z, fj, v[c].z);
        v[c].w = fmaf(e[c].w, fj, v[c].w);
      }
  };
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    if (bias != nullptr && col < W) {
      v[c].x += Elem<T>::get(bias[col]);
      if (VEC || col + 1 < W) v[c].y += Elem<T>::get(bias[col + 1]);
      if (VEC || col + 2 < W) v[c].z += Elem<T>::get(bias[col + 2]);
      if (VEC || col + 3 < W) v[c].w += Elem<T>::get(bias[col + 3]);
    }
    v[c].x *= fy;
    v[c].y *= fy;
    v[c].z *= fy;
    v[c].w *= fy;
  }
#pragma unroll
  for (int j = 0; j < PN_TOP; ++j) add(r[j], f[j]);
  for (int j = PN_TOP; j < p.top; ++j) add(p.row_of[row * p.top + j], p.mix != nullptr ? p.mix[row * p.top + j] : 1.f / float(p.top));
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    if (!VEC) {
      const int col = col_of(c);
      if (col + 1 >= W) v[c].y = 0.f;
      if (col + 2 >= W) v[c].z = 0.f;
      if (col + 3 >= W) v[c].w = 0.f;
    }
    ss += v[c].x * v[c].x + v[c].y * v[c].y + v[c].z * v[c].z + v[c].w * v[c].w;
  }
  const float inv = rsqrtf(cta_sum<PN_THREADS>(ss, red) / float(W) + p.eps);
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    if (col >= W) continue;
    if (VEC) {
      const float4 w = *reinterpret_cast<const float4*>(p.w + col);
      const float4 n = make_float4(xv[c].x + v[c].x * inv * w.x, xv[c].y + v[c].y * inv * w.y, xv[c].z + v[c].z * inv * w.z,
                                   xv[c].w + v[c].w * inv * w.w);
      *reinterpret_cast<float4*>(x + col) = n;
      store4(h + col, n.x, n.y, n.z, n.w);
    } else {
      const float a[4] = {v[c].x, v[c].y, v[c].z, v[c].w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (col + i >= W) break;
        const float n = x[col + i] + a[i] * inv * p.w[col + i];
        x[col + i] = n;
        h[col + i] = Elem<T>::put(n);
      }
    }
  }
  for (int c = W + threadIdx.x; c < p.Wp; c += PN_THREADS) h[c] = Elem<T>::put(0.f);
}

// The same for many rows of finished projections (bf16, W a multiple of 4, at most TOP expert rows per token): a CTA walks rows
// and has the next one's loads in flight while it norms and writes this one
template <int NC, int TOP>
__global__ void __launch_bounds__(PN_THREADS, NC <= 2 ? 2 : 1)
post_norm_rows_kernel(const PostNormAdd p) {
  constexpr int E = TOP > 0 ? TOP : 1;
  __shared__ float red[2][PN_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int W = p.W, tid = threadIdx.x, step = gridDim.x;
  auto col_of = [&](int c) { return (tid + c * PN_THREADS) * 4; };
  const bf16 *y = reinterpret_cast<const bf16*>(p.y.p), *ey = reinterpret_cast<const bf16*>(p.experts.p);
  uint2 y4[NC], e4[E][NC];
  float4 x4[NC];
  int r[E];
  float f[E], fn[E], fy = 1.f;                               // factors of this row; of the next one
  auto index = [&](int row) {
#pragma unroll
    for (int j = 0; j < TOP; ++j) {
      const bool on = row < p.T && j < p.top;
      r[j] = on ? p.row_of[row * p.top + j] : -1;
      fn[j] = !on ? 0.f : p.mix != nullptr ? p.mix[row * p.top + j] : 1.f / float(p.top);
    }
  };
  auto request = [&](int row) {                              // index(row) is there
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int col = col_of(c);
      if (col >= W) continue;
      y4[c] = __ldcg(reinterpret_cast<const uint2*>(y + row * p.y.ld + col));
      x4[c] = __ldcg(reinterpret_cast<const float4*>(p.x + (long long)row * W + col));
#pragma unroll
      for (int j = 0; j < TOP; ++j)
        e4[j][c] = r[j] >= 0 ? __ldcg(reinterpret_cast<const uint2*>(ey + r[j] * p.experts.ld + col)) : make_uint2(0, 0);
    }
    if (p.y_factor != nullptr) fy = p.y_factor[row];
#pragma unroll
    for (int j = 0; j < TOP; ++j) f[j] = fn[j];
  };
  auto wide = [](const uint2& u) {
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                       __uint_as_float(u.y & 0xffff0000u));
  };
  int row = blockIdx.x;
  index(row);
  if (row < p.T) request(row);
  index(row + step);
  for (int par = 0; row < p.T; row += step, par ^= 1) {
    float4 v[NC], x[NC];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      v[c] = x[c] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (col_of(c) >= W) continue;
      const float4 a = wide(y4[c]);
      v[c] = make_float4(a.x * fy, a.y * fy, a.z * fy, a.w * fy);
#pragma unroll
      for (int j = 0; j < TOP; ++j) {
        const float4 e = wide(e4[j][c]);
        v[c].x = fmaf(e.x, f[j], v[c].x);
        v[c].y = fmaf(e.y, f[j], v[c].y);
        v[c].z = fmaf(e.z, f[j], v[c].z);
        v[c].w = fmaf(e.w, f[j], v[c].w);
      }
      x[c] = x4[c];
      ss += v[c].x * v[c].x + v[c].y * v[c].y + v[c].z * v[c].z + v[c].w * v[c].w;
    }
    if (row + step < p.T) {
      request(row + step);
      index(row + 2 * step);
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[par][tid >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < PN_THREADS / 32; ++i) ss += red[par][i];
    const float inv = rsqrtf(ss / float(W) + p.eps);
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int col = col_of(c);
      if (col >= W) continue;
      const float4 w = *reinterpret_cast<const float4*>(p.w + col);
      const float4 n = make_float4(x[c].x + v[c].x * inv * w.x, x[c].y + v[c].y * inv * w.y, x[c].z + v[c].z * inv * w.z,
                                   x[c].w + v[c].w * inv * w.w);
      *reinterpret_cast<float4*>(p.x + (long long)row * W + col) = n;
      store4(reinterpret_cast<bf16*>(p.h) + (long long)row * p.Wp + col, n.x, n.y, n.z, n.w);
    }
    if (tid < p.Wp - W) reinterpret_cast<bf16*>(p.h)[(long long)row * p.Wp + W + tid] = __float2bfloat16(0.f);
  }
}
static bool post_norm_rows(const PostNormAdd& p, cudaStream_t s) {
  if (p.T < 1024 || p.W % 4 != 0 || !p.has_y || p.y.part != nullptr || p.bias != nullptr || p.top > 4 ||
      (p.top > 0 && p.experts.part != nullptr))
    return false;
  auto go = [&](auto kern, int ctas) { launch_pdl(PDL_NORM, kern, dim3(148 * ctas), dim3(PN_THREADS), 0, s, p); };
  auto pick = [&](auto nc) {
    constexpr int NC = decltype(nc)::value;
    constexpr int ctas = NC <= 2 ? 2 : 1;
    if (p.top == 0) go(post_norm_rows_kernel<NC, 0>, ctas);
    else if (p.top <= 2) go(post_norm_rows_kernel<NC, 2>, ctas);
    else go(post_norm_rows_kernel<NC, 4>, ctas);
  };
  if (p.W <= PN_THREADS * 4) pick(std::integral_constant<int, 1>{});
  else if (p.W <= PN_THREADS * 8) pick(std::integral_constant<int, 2>{});
  else pick(std::integral_constant<int, 4>{});
  return true;
}

// x (+)= y + mixed expert rows;  h = rms(x) * w (or x) in the model's type, zero-padded from W to Wp columns.  NC: 4-column
// chunks per thread
template <typename T, bool VEC, int NC>
__global__ void __launch_bounds__(RS_THREADS)
add_norm_kernel(const AddNorm p, const ProjSrc y, int has_y) {
  __shared__ float red[RS_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  const int W = p.W;
  float* x = p.x + row * W;
  T* h = reinterpret_cast<T*>(p.h) + row * p.ld_h;
  auto col_of = [&](int c) { return (int(threadIdx.x) + c * RS_THREADS) * 4; };
  float4 v[NC];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    v[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!p.add || col >= W) continue;
    if (VEC) {
      v[c] = __ldcg(reinterpret_cast<const float4*>(x + col));
    } else {
      v[c].x = x[col];
      if (col + 1 < W) v[c].y = x[col + 1];
      if (col + 2 < W) v[c].z = x[col + 2];
      if (col + 3 < W) v[c].w = x[col + 3];
    }
  }
  auto add4 = [&](int c, const float4& a, float f) {
    v[c].x = fmaf(a.x, f, v[c].x);
    v[c].y = fmaf(a.y, f, v[c].y);
    v[c].z = fmaf(a.z, f, v[c].z);
    v[c].w = fmaf(a.w, f, v[c].w);
  };
  if (has_y)
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (col_of(c) < W) add4(c, proj_at4<T>(y, row, col_of(c)), 1.f);     // pad columns of a projection exist and are zero
  for (int j = 0; j < p.top; ++j) {
    const int r = p.row_of[row * p.top + j];
    if (r < 0) continue;
    const float f = p.mix != nullptr ? p.mix[row * p.top + j] : 1.f / float(p.top);
    float4 e[NC];
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (col_of(c) < W) e[c] = proj_at4<T>(p.experts, r, col_of(c));
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (col_of(c) < W) add4(c, e[c], f);
  }
  const bool changed = has_y || p.top > 0;
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    if (col >= W) continue;
    if (VEC) {
      if (changed) *reinterpret_cast<float4*>(x + col) = v[c];
    } else {
      if (col + 1 >= W) v[c].y = 0.f;
      if (col + 2 >= W) v[c].z = 0.f;
      if (col + 3 >= W) v[c].w = 0.f;
      x[col] = v[c].x;
      if (col + 1 < W) x[col + 1] = v[c].y;
      if (col + 2 < W) x[col + 2] = v[c].z;
      if (col + 3 < W) x[col + 3] = v[c].w;
    }
    ss += v[c].x * v[c].x + v[c].y * v[c].y + v[c].z * v[c].z + v[c].w * v[c].w;
  }
  const bool norm = p.w != nullptr;
  const float inv = norm ? rsqrtf(cta_sum<RS_THREADS>(ss, red) / float(W) + p.eps) : 1.f;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    if (col >= W) continue;
    if (VEC) {
      const float4 w = norm ? *reinterpret_cast<const float4*>(p.w + col) : make_float4(1.f, 1.f, 1.f, 1.f);
      store4(h + col, v[c].x * inv * w.x, v[c].y * inv * w.y, v[c].z * inv * w.z, v[c].w * inv * w.w);
    } else {
      const float a[4] = {v[c].x, v[c].y, v[c].z, v[c].w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (col + i < W) h[col + i] = Elem<T>::put(a[i] * inv * (norm ? p.w[col + i] : 1.f));
    }
  }
  for (int c = W + threadIdx.x; c < p.Wp; c += RS_THREADS) h[c] = Elem<T>::put(0.f);
}

// eight columns per thread, grid as gelu_mul_kernel
template <typename T, int KIND>
__global__ void __launch_bounds__(RS_THREADS)
glu_mul_kernel(const GluMul a) {
  pdl_launch_dependents();
  pdl_wait();
  const int col = (blockIdx.x * RS_THREADS + threadIdx.x) * 8;
  if (col >= a.width_p) return;
#pragma unroll 2
  for (int row = blockIdx.y; row < a.T; row += gridDim.y) {
    float g[8], u[8], o[8];
    proj_at8<T>(a.p, row, a.off_gate + col, g);
    proj_at8<T>(a.p, row, a.off_up + col, u);
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = col + j < a.width ? glu_t<T, KIND>(g[j], u[j], a.limit) : 0.f;
    store8(reinterpret_cast<T*>(a.out) + row * a.ld_out + col, o);
  }
}

// the same grid; one input
template <typename T>
__global__ void __launch_bounds__(RS_THREADS)
xielu_kernel(const ProjSrc z, const float* __restrict__ coef, T* __restrict__ out, int rows, int width, int width_p) {
  pdl_launch_dependents();
  pdl_wait();
  const int col = (blockIdx.x * RS_THREADS + threadIdx.x) * 8;
  if (col >= width_p) return;
  const float a = coef[0], b = coef[1];
#pragma unroll 2
  for (int row = blockIdx.y; row < rows; row += gridDim.y) {
    float v[8];
    proj_at8<T>(z, row, col, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = col + j < width ? xielu_t<T>(v[j], a, b) : 0.f;
    store8(out + (long long)row * width_p + col, v);
  }
}

template <typename T>
__global__ void __launch_bounds__(RS_THREADS)
rms_norm_wide_kernel(const float* __restrict__ x, const float* __restrict__ w, T* __restrict__ h, int W, int Wp,
                     float eps) {
  __shared__ float red[RS_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  float ss = 0.f;
  for (int c = threadIdx.x; c < W; c += RS_THREADS) {
    const float v = x[row * W + c];
    ss += v * v;
  }
  const float inv = rsqrtf(cta_sum<RS_THREADS>(ss, red) / float(W) + eps);
  for (int c = threadIdx.x; c < Wp; c += RS_THREADS)
    h[row * Wp + c] = Elem<T>::put(c < W ? x[row * W + c] * inv * w[c] : 0.f);
}

// out = gelu_tanh(gate + bias) * (up + bias), eight columns per thread; grid (column blocks, row groups)
template <typename T>
__global__ void __launch_bounds__(RS_THREADS)
gelu_mul_kernel(const ProjSrc gu, const T* __restrict__ bias, T* __restrict__ out, int rows, int up_off, int width,
                int width_p) {
  pdl_launch_dependents();
  pdl_wait();
  const int col = (blockIdx.x * RS_THREADS + threadIdx.x) * 8;
  if (col >= width_p) return;
  float bg[8], bu[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    bg[j] = bias != nullptr ? Elem<T>::get(bias[col + j]) : 0.f;
    bu[j] = bias != nullptr ? Elem<T>::get(bias[up_off + col + j]) : 0.f;
  }
#pragma unroll 2
  for (int row = blockIdx.y; row < rows; row += gridDim.y) {
    float g[8], u[8], o[8];
    proj_at8<T>(gu, row, col, g);
    proj_at8<T>(gu, row, up_off + col, u);
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = col + j < width ? gelu_tanh_t<T>(g[j] + bg[j]) * (u[j] + bu[j]) : 0.f;
    store8(out + (long long)row * width_p + col, o);
  }
}

// ================================================================= launchers
static void check_launch(const char* what) {
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string(what) + ": " + cudaGetErrorString(e));
}

template <typename T>
static void embed_t(const void* ids, const void* weight, float* x, void* h, int T_, int W, int Wp, long long V,
                    float scale, uint32_t* status, cudaStream_t s) {
  launch_pdl(PDL_EMBEDDING, embed_scaled_kernel<T>, dim3(T_), dim3(RS_THREADS), 0, s, (const long long*)ids,
             (const T*)weight, x, (T*)h, W, Wp, V, scale, status);
}
void launch_embed_scaled(const void* ids, const void* weight, float* x, void* h, int T, int W, int Wp, long long V,
                         float scale, bool f32, uint32_t* status, cudaStream_t s) {
  if (T == 0) return;
  if (f32) embed_t<float>(ids, weight, x, h, T, W, Wp, V, scale, status, s);
  else embed_t<bf16>(ids, weight, x, h, T, W, Wp, V, scale, status, s);
  check_launch("embedding");
}

void launch_post_norm_add(const PostNormAdd& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (p.W > PN_THREADS * 16) throw std::runtime_error("norm rows are limited to 8192 columns");
  auto go = [&](auto kern) { launch_pdl(PDL_NORM, kern, dim3(p.T), dim3(PN_THREADS), 0, s, p); };
  if (!f32 && post_norm_rows(p, s)) {
  } else if (p.W % 4 != 0) {
    if (f32) go(post_norm_add_kernel<float, false, 4>);
    else go(post_norm_add_kernel<bf16, false, 4>);
  } else if (f32) {
    go(post_norm_add_kernel<float, true, 4>);
  } else if (p.W <= PN_THREADS * 4) {
    go(post_norm_add_kernel<bf16, true, 1>);
  } else if (p.W <= PN_THREADS * 8) {
    go(post_norm_add_kernel<bf16, true, 2>);
  } else {
    go(post_norm_add_kernel<bf16, true, 4>);
  }
  check_launch("norm + add");
}

void launch_rms_norm_wide(const float* x, const float* w, void* h, int T, int W, int Wp, float eps, bool f32,
                          cudaStream_t s) {
  if (T == 0) return;
  if (f32)
    launch_pdl(PDL_NORM, rms_norm_wide_kernel<float>, dim3(T), dim3(RS_THREADS), 0, s, x, w, (float*)h, W, Wp, eps);
  else
    launch_pdl(PDL_NORM, rms_norm_wide_kernel<bf16>, dim3(T), dim3(RS_THREADS), 0, s, x, w, (bf16*)h, W, Wp, eps);
  check_launch("final norm");
}

void launch_add_norm(const AddNorm& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (p.W > RS_THREADS * RS_CHUNKS * 4) throw std::runtime_error("norm rows are limited to 8192 columns");
  const ProjSrc y = p.y != nullptr ? *p.y : ProjSrc();
  const int has_y = p.y != nullptr ? 1 : 0;
  auto go = [&](auto kern) { launch_pdl(PDL_NORM, kern, dim3(p.T), dim3(RS_THREADS), 0, s, p, y, has_y); };
  const int chunks = (p.W + RS_THREADS * 4 - 1) / (RS_THREADS * 4);
  if (p.W % 4 != 0) {
    if (f32) go(add_norm_kernel<float, false, RS_CHUNKS>);
    else go(add_norm_kernel<bf16, false, RS_CHUNKS>);
  } else if (f32) {
    go(add_norm_kernel<float, true, RS_CHUNKS>);
  } else if (chunks <= 2) {
    go(add_norm_kernel<bf16, true, 2>);
  } else if (chunks <= 4) {
    go(add_norm_kernel<bf16, true, 4>);
  } else {
    go(add_norm_kernel<bf16, true, RS_CHUNKS>);
  }
  check_launch("add + norm");
}

void launch_glu_mul(const GluMul& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  const int cols = (p.width_p / 8 + RS_THREADS - 1) / RS_THREADS;
  const dim3 grid(cols, std::min(p.T, std::max(1, 148 * 8 / cols)));
  auto go = [&](auto kern) { launch_pdl(PDL_PARTIALS, kern, grid, dim3(RS_THREADS), 0, s, p); };
  if (p.kind == GLU_ACT_SILU) {
    if (f32) go(glu_mul_kernel<float, GLU_ACT_SILU>);
    else go(glu_mul_kernel<bf16, GLU_ACT_SILU>);
  } else {
    if (f32) go(glu_mul_kernel<float, GLU_ACT_CLAMPED>);
    else go(glu_mul_kernel<bf16, GLU_ACT_CLAMPED>);
  }
  check_launch("gated activation");
}

void launch_xielu(const ProjSrc& z, const float* c, void* out, int T, int width, int width_p, bool f32, cudaStream_t s) {
  if (T == 0) return;
  const int cols = (width_p / 8 + RS_THREADS - 1) / RS_THREADS;
  const dim3 grid(cols, std::min(T, std::max(1, 148 * 8 / cols)));
  if (f32) launch_pdl(PDL_PARTIALS, xielu_kernel<float>, grid, dim3(RS_THREADS), 0, s, z, c, (float*)out, T, width, width_p);
  else launch_pdl(PDL_PARTIALS, xielu_kernel<bf16>, grid, dim3(RS_THREADS), 0, s, z, c, (bf16*)out, T, width, width_p);
  check_launch("xIELU");
}

void launch_gelu_mul(const ProjSrc& gu, const void* bias, void* out, int T, int up_off, int width, int width_p,
                     bool f32, cudaStream_t s) {
  if (T == 0) return;
  const int cols = (width_p / 8 + RS_THREADS - 1) / RS_THREADS;
  const dim3 grid(cols, std::min(T, std::max(1, 148 * 8 / cols)));
  if (f32)
    launch_pdl(PDL_PARTIALS, gelu_mul_kernel<float>, grid, dim3(RS_THREADS), 0, s, gu, (const float*)bias, (float*)out, T,
               up_off, width, width_p);
  else
    launch_pdl(PDL_PARTIALS, gelu_mul_kernel<bf16>, grid, dim3(RS_THREADS), 0, s, gu, (const bf16*)bias, (bf16*)out, T,
               up_off, width, width_p);
  check_launch("gelu gate");
}

}  // namespace fc
