// Several fp32 residual streams (hyper-connections): a sublayer's output is spread over the streams while they are mixed, and
// the next sublayer's input, the layer norm of a weighted sum of the new streams, is made in the same pass.  One CTA per
// token; a thread owns columns of all streams, so that each is read and written once.
#include <stdexcept>
#include <string>

#include "hybrid.cuh"
#include "launch.h"

namespace fc {

using bf16 = __nv_bfloat16;

// four columns of a row of W (VEC: W is a multiple of 4)
template <bool VEC>
__device__ __forceinline__ float4 row_get4(const float* __restrict__ row, int col, int W) {
  if (VEC) return __ldcg(reinterpret_cast<const float4*>(row + col));
  float4 v = make_float4(row[col], 0.f, 0.f, 0.f);
  if (col + 1 < W) v.y = row[col + 1];
  if (col + 2 < W) v.z = row[col + 2];
  if (col + 3 < W) v.w = row[col + 3];
  return v;
}
template <bool VEC>
__device__ __forceinline__ void row_put4(float* __restrict__ row, int col, int W, const float4& v) {
  if (VEC) {
    *reinterpret_cast<float4*>(row + col) = v;
    return;
  }
  row[col] = v.x;
  if (col + 1 < W) row[col + 1] = v.y;
  if (col + 2 < W) row[col + 2] = v.z;
  if (col + 3 < W) row[col + 3] = v.w;
}
__device__ __forceinline__ void axpy4(float4& d, float f, const float4& a) {
  d.x = fmaf(f, a.x, d.x);
  d.y = fmaf(f, a.y, d.y);
  d.z = fmaf(f, a.z, d.z);
  d.w = fmaf(f, a.w, d.w);
}

// h = (u - mean) / sqrt(var + eps) * w + b of the row whose columns u the CTA's threads hold; columns [W, Wp) are zeroed
template <typename T, bool VEC, int NC, int THREADS>
__device__ __forceinline__ void put_layer_norm(const StreamMix& p, long long row, float4 (&u)[NC], float* red) {
  auto col_of = [&](int c) { return (int(threadIdx.x) + c * THREADS) * 4; };
  float s = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c)
    if (col_of(c) < p.W) s += u[c].x + u[c].y + u[c].z + u[c].w;        // columns past W hold zeros
  const float mean = cta_sum<THREADS>(s, red) / float(p.W);
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    if (col >= p.W) continue;
    u[c].x -= mean;
    u[c].y -= mean;
    u[c].z -= mean;
    u[c].w -= mean;
    if (!VEC) {
      if (col + 1 >= p.W) u[c].y = 0.f;
      if (col + 2 >= p.W) u[c].z = 0.f;
      if (col + 3 >= p.W) u[c].w = 0.f;
    }
    ss += u[c].x * u[c].x + u[c].y * u[c].y + u[c].z * u[c].z + u[c].w * u[c].w;
  }
  const float inv = rsqrtf(cta_sum<THREADS>(ss, red) / float(p.W) + p.eps);
  T* h = reinterpret_cast<T*>(p.h) + row * p.ld_h;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    if (col >= p.W) continue;
    const float4 w = row_get4<VEC>(p.w, col, p.W), b = row_get4<VEC>(p.b, col, p.W);
    const float o[4] = {fmaf(u[c].x * inv, w.x, b.x), fmaf(u[c].y * inv, w.y, b.y), fmaf(u[c].z * inv, w.z, b.z),
                        fmaf(u[c].w * inv, w.w, b.w)};
    if (VEC) {
      store4(h + col, o[0], o[1], o[2], o[3]);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (col + i < p.W) h[col + i] = Elem<T>::put(o[i]);
    }
  }
  for (int c = p.W + threadIdx.x; c < p.Wp; c += THREADS) h[c] = Elem<T>::put(0.f);
}

// SM: most streams of this instance (p.S of them exist)
template <typename T, bool VEC, int NC, int SM, int THREADS>
__global__ void __launch_bounds__(THREADS)
stream_mix_kernel(const StreamMix p) {
  __shared__ float red[THREADS / 32];
  float in[SM], out[SM], mix[SM][SM];                       // parameters: no kernel writes them
#pragma unroll
  for (int s = 0; s < SM; ++s) {
    const bool on = s < p.S;
    in[s] = on ? (p.next != nullptr ? p.next[s] : 1.f) : 0.f;
    out[s] = on ? p.connection[p.S + s] : 0.f;
#pragma unroll
    for (int t = 0; t < SM; ++t) mix[s][t] = on && t < p.S ? p.connection[2 * p.S + s * p.S + t] : 0.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  const int W = p.W;
  auto col_of = [&](int c) { return (int(threadIdx.x) + c * THREADS) * 4; };
  float4 u[NC];
  if (p.has_y) {
#pragma unroll
    for (int c = 0; c < NC; ++c)
      u[c] = col_of(c) < W ? proj_at4<T>(p.y, row, col_of(c)) : make_float4(0.f, 0.f, 0.f, 0.f);
  } else {
#pragma unroll
    for (int c = 0; c < NC; ++c) u[c] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int j = 0; j < p.top; ++j) {
    const int r = __ldcg(p.row_of + row * p.top + j);
    if (r < 0) continue;
    const float f = p.mix != nullptr ? __ldcg(p.mix + row * p.top + j) : 1.f / float(p.top);
    float4 e[NC];
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (col_of(c) < W) e[c] = proj_at4<T>(p.experts, r, col_of(c));
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (col_of(c) < W) axpy4(u[c], f, e[c]);
  }
  float* x = p.x + row * p.S * W;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = col_of(c);
    if (col >= W) continue;
    const float4 y = u[c];
    float4 old[SM];
#pragma unroll
    for (int s = 0; s < SM; ++s) old[s] = s < p.S ? row_get4<VEC>(x + s * W, col, W) : make_float4(0.f, 0.f, 0.f, 0.f);
    u[c] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int t = 0; t < SM; ++t) {
      if (t >= p.S) break;
      float4 v = make_float4(out[t] * y.x, out[t] * y.y, out[t] * y.z, out[t] * y.w);
#pragma unroll
      for (int s = 0; s < SM; ++s) axpy4(v, mix[s][t], old[s]);
      if (p.next != nullptr) row_put4<VEC>(x + t * W, col, W, v);
      axpy4(u[c], in[t], v);
    }
    if (!VEC) {                                             // what a projection's pad columns may add
      if (col + 1 >= W) u[c].y = 0.f;
      if (col + 2 >= W) u[c].z = 0.f;
      if (col + 3 >= W) u[c].w = 0.f;
    }
  }
  put_layer_norm<T, VEC, NC, THREADS>(p, row, u, red);
}

// the streams at the start: all the row of the table
template <typename T, bool VEC, int NC, int THREADS>
__global__ void __launch_bounds__(THREADS)
embed_streams_kernel(const StreamMix p, const long long* __restrict__ ids, const T* __restrict__ table, long long vocab,
                     uint32_t* status) {
  __shared__ float red[THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  long long id = ids[row];
  const bool ok = id >= 0 && id < vocab;
  if (!ok) {
    if (threadIdx.x == 0) report(status, ST_BAD_INDEX);
    id = 0;
  }
  float sum = 0.f;
  for (int s = 0; s < p.S; ++s) sum += p.next != nullptr ? p.next[s] : 1.f;
  float4 u[NC];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = (int(threadIdx.x) + c * THREADS) * 4;
    u[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (col >= p.W) continue;
    const T* e = table + id * p.Wp + col;                   // the table's rows are padded to whole 8 columns with zeros
    if (ok) u[c] = make_float4(Elem<T>::get(e[0]), Elem<T>::get(e[1]), Elem<T>::get(e[2]), Elem<T>::get(e[3]));
    for (int s = 0; s < p.S; ++s) row_put4<VEC>(p.x + (row * p.S + s) * p.W, col, p.W, u[c]);
    u[c] = make_float4(u[c].x * sum, u[c].y * sum, u[c].z * sum, u[c].w * sum);
  }
  put_layer_norm<T, VEC, NC, THREADS>(p, row, u, red);
}

// ================================================================= launchers
static void check_launch(const char* what) {
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string(what) + ": " + cudaGetErrorString(e));
}
static void check_sizes(const StreamMix& p) {
  if (p.W > STREAM_MAX_WIDTH) throw std::runtime_error("norm rows are limited to 8192 columns");
  if (p.S < 1 || p.S > STREAM_MAX) throw std::runtime_error("residual streams are limited to 16");
}

template <typename T>
static void stream_mix_t(const StreamMix& p, cudaStream_t s) {
  auto go = [&](auto kern, int threads) { launch_pdl(PDL_NORM, kern, dim3(p.T), dim3(threads), 0, s, p); };
  const bool vec = p.W % 4 == 0;
  if (!vec || p.S > 4) {
    if (p.S > 8) {
      if (vec) go(stream_mix_kernel<T, true, 8, 16, 256>, 256);
      else go(stream_mix_kernel<T, false, 8, 16, 256>, 256);
    } else {
      if (vec) go(stream_mix_kernel<T, true, 8, 8, 256>, 256);
      else go(stream_mix_kernel<T, false, 8, 8, 256>, 256);
    }
    return;
  }
  const int chunks = (p.W + 1023) / 1024;
  auto pick = [&](auto sm) {
    constexpr int SM = decltype(sm)::value;
    if (p.T <= 296) {                                       // few rows: more threads per row
      if (p.W <= 4096) go(stream_mix_kernel<T, true, 1, SM, 1024>, 1024);
      else go(stream_mix_kernel<T, true, 2, SM, 1024>, 1024);
    } else if (chunks <= 1) {
      go(stream_mix_kernel<T, true, 1, SM, 256>, 256);
    } else if (chunks <= 2) {
      go(stream_mix_kernel<T, true, 2, SM, 256>, 256);
    } else if (chunks <= 4) {
      go(stream_mix_kernel<T, true, 4, SM, 256>, 256);
    } else {
      go(stream_mix_kernel<T, true, 8, SM, 256>, 256);
    }
  };
  if (p.S == 1) pick(std::integral_constant<int, 1>{});
  else if (p.S == 2) pick(std::integral_constant<int, 2>{});
  else pick(std::integral_constant<int, 4>{});
}
void launch_stream_mix(const StreamMix& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  check_sizes(p);
  if (f32) stream_mix_t<float>(p, s);
  else stream_mix_t<bf16>(p, s);
  check_launch("mix of the residual streams");
}

template <typename T>
static void embed_t(const StreamMix& p, const void* ids, const void* table, long long vocab, uint32_t* status, cudaStream_t s) {
  auto go = [&](auto kern) {
    launch_pdl(PDL_EMBEDDING, kern, dim3(p.T), dim3(256), 0, s, p, (const long long*)ids, (const T*)table, vocab, status);
  };
  if (p.W % 4 != 0) go(embed_streams_kernel<T, false, 8, 256>);
  else if (p.W <= 2048) go(embed_streams_kernel<T, true, 2, 256>);
  else go(embed_streams_kernel<T, true, 8, 256>);
}
void launch_embed_streams(const StreamMix& p, const void* ids, const void* table, long long vocab, bool f32, uint32_t* status,
                          cudaStream_t s) {
  if (p.T == 0) return;
  check_sizes(p);
  if (f32) embed_t<float>(p, ids, table, vocab, status, s);
  else embed_t<bf16>(p, ids, table, vocab, status, s);
  check_launch("embedding of the residual streams");
}

}  // namespace fc
