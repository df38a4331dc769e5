// Device helpers of the hybrid-model kernels: element type conversion and reads of projection outputs.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "hybrid.h"
#include "ptx.cuh"

namespace fc {

template <typename T>
struct Elem;
template <>
struct Elem<float> {
  static __device__ __forceinline__ float get(float v) { return v; }
  static __device__ __forceinline__ float put(float v) { return v; }
};
template <>
struct Elem<__nv_bfloat16> {
  static __device__ __forceinline__ float get(__nv_bfloat16 v) { return __bfloat162float(v); }
  static __device__ __forceinline__ __nv_bfloat16 put(float v) { return __float2bfloat16(v); }
};

// one element of a projection output
template <typename T>
__device__ __forceinline__ float proj_at(const ProjSrc& s, long long row, int col) {
  if (s.part != nullptr) {
    float v = 0.f;
    const float* p = s.part + row * s.part_ld + col;
    for (int i = 0; i < s.splits; ++i) v += __ldcg(p + i * s.part_stride);
    return v;
  }
  return Elem<T>::get(reinterpret_cast<const T*>(s.p)[row * s.ld + col]);
}

// four consecutive elements; `col` and the pitches are multiples of 4
template <typename T>
__device__ __forceinline__ float4 proj_at4(const ProjSrc& s, long long row, int col) {
  if (s.part != nullptr) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    const float* p = s.part + row * s.part_ld + col;
#pragma unroll 4
    for (int i = 0; i < s.splits; ++i) {
      const float4 a = __ldcg(reinterpret_cast<const float4*>(p + i * s.part_stride));
      v.x += a.x;
      v.y += a.y;
      v.z += a.z;
      v.w += a.w;
    }
    return v;
  }
  const T* q = reinterpret_cast<const T*>(s.p) + row * s.ld + col;
  if constexpr (sizeof(T) == 4) {
    return __ldcg(reinterpret_cast<const float4*>(q));
  } else {
    const uint2 u = __ldcg(reinterpret_cast<const uint2*>(q));
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
  }
}

template <typename T>
__device__ __forceinline__ void store4(T* dst, float a, float b, float c, float d) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
  } else {
    uint2 u;
    u.x = pack_bf16(a, b);
    u.y = pack_bf16(c, d);
    *reinterpret_cast<uint2*>(dst) = u;
  }
}

// eight consecutive elements; `col` and the pitches are multiples of 8
template <typename T>
__device__ __forceinline__ void proj_at8(const ProjSrc& s, long long row, int col, float (&v)[8]) {
  if (sizeof(T) == 2 && s.part == nullptr) {
    const uint4 u = __ldcg(reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(s.p) + row * s.ld + col));
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
    return;
  }
  const float4 a = proj_at4<T>(s, row, col), b = proj_at4<T>(s, row, col + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <typename T>
__device__ __forceinline__ void store8(T* dst, const float (&v)[8]) {
  if constexpr (sizeof(T) == 2) {
    *reinterpret_cast<uint4*>(dst) =
        make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  } else {
    store4(dst, v[0], v[1], v[2], v[3]);
    store4(dst + 4, v[4], v[5], v[6], v[7]);
  }
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// activations of a model in T: the fast intrinsics where the result is rounded to bf16 anyway
template <typename T>
__device__ __forceinline__ float over_one_plus_exp(float x, float e) {      // x / (1 + exp(e))
  if constexpr (sizeof(T) == 2) return __fdividef(x, 1.f + __expf(e));
  return x / (1.f + expf(e));
}
template <typename T>
__device__ __forceinline__ float silu_t(float x) { return over_one_plus_exp<T>(x, -x); }
template <typename T>
__device__ __forceinline__ float sigmoid_t(float x) { return over_one_plus_exp<T>(1.f, -x); }
// log(sigmoid(x)) and log(1 + exp(x)) without overflow
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// 0.5 z (1 + tanh y) = z sigmoid(2 y) with y = sqrt(2 / pi) (z + 0.044715 z^3)
template <typename T>
__device__ __forceinline__ float gelu_tanh_t(float z) {
  return over_one_plus_exp<T>(z, -1.5957691216057308f * (z + 0.044715f * z * z * z));
}

// gated activations (GluKind)
template <typename T, int KIND>
__device__ __forceinline__ float glu_t(float g, float u, float limit) {
  if (KIND == GLU_ACT_SILU) return silu_t<T>(g) * u;
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return over_one_plus_exp<T>(g, -1.702f * g) * (u + 1.f);
}

// xIELU: z > 0: a z^2 + z / 2, else b (e^z - 1 - z) + z / 2.  e^z - 1 - z cancels near 0: its series there
template <typename T>
__device__ __forceinline__ float xielu_t(float z, float a, float b) {
  const float n = fminf(z, 0.f);
  float e;
  if constexpr (sizeof(T) == 2) {
    e = __expf(n) - 1.f - n;
    if (n > -0.0625f) e = n * n * (0.5f + n * (0.16666667f + n * 0.041666667f));
  } else {
    e = expm1f(n) - n;
    if (n > -0.25f) e = n * n * (0.5f + n * (0.16666667f + n * (0.041666667f + n * (0.0083333333f + n * 0.0013888889f))));
  }
  return (z > 0.f ? a * z * z : b * e) + 0.5f * z;
}

// cos and sin of `position` times a frequency in turns: reduced in double, so that far positions lose nothing
__device__ __forceinline__ void turn_angle(double pos, double freq, float& c, float& s) {
  const double turns = pos * freq;
  sincospif(float(2.0 * (turns - rint(turns))), &s, &c);
}

struct Run {
  int lo, len, start, slot;
};
__device__ __forceinline__ Run get_run(const RunBatch& r, int b) {
  Run o;
  o.lo = r.cu != nullptr ? r.cu[b] : b;
  o.len = r.cu != nullptr ? r.cu[b + 1] - o.lo : 1;
  const int n = r.ctx[b];
  o.slot = r.slots[b];
  o.start = n - o.len;
  if (n <= 0 || o.slot < 0 || o.slot >= r.num_slots) o.slot = -1;
  return o;
}

template <int THREADS>
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) t += red[i];
  __syncthreads();
  return t;
}

}  // namespace fc
