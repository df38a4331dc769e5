// Device side of AttnOptions: the first visible key of a query, the soft cap of scores.
#pragma once
#include "kernels.h"
#include "ptx.cuh"

namespace fc {

constexpr float ATTN_LOG2E = 1.4426950408889634f;

// first key that the query at position `pos` sees
__device__ __forceinline__ int attn_first(const AttnOptions& o, int pos) {
  int first = o.window > 0 ? max(0, pos - o.window + 1) : 0;
  if (o.chunk > 0) first = max(first, pos - pos % o.chunk);
  return first;
}

// tanh by exponential and reciprocal: error about 1e-7 of the full range
__device__ __forceinline__ float tanh_exp(float x) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(fminf(x, 20.f) * (2.f * ATTN_LOG2E)));
  return 1.f - __fdividef(2.f, 1.f + e);
}
// tanh for |x| <= TANH_POLY_MAX without a special-function instruction: x p(x^2), p the Chebyshev interpolant of degree 5
// of tanh(sqrt z) / sqrt z on [0, TANH_POLY_MAX^2] (error 4e-8)
constexpr float TANH_POLY_MAX = 0.8f;
__device__ __forceinline__ float tanh_poly(float x) {
  const float z = x * x;
  float p = -0.0043497388f;
  p = fmaf(p, z, 0.019084353f);
  p = fmaf(p, z, -0.05310927f);
  p = fmaf(p, z, 0.13320932f);
  p = fmaf(p, z, -0.33332667f);
  p = fmaf(p, z, 0.99999994f);
  return x * p;
}

// raw dot products to scores in log2 units: s * scale_log2, or capped (in = scale / cap, out = cap * log2 e)
struct ScoreScale {
  float scale_log2, in, out;
  bool cap;
};
__device__ __forceinline__ ScoreScale score_scale(const AttnOptions& o, float scale_log2) {
  ScoreScale r;
  r.scale_log2 = scale_log2;
  r.cap = o.softcap > 0.f;
  r.in = r.cap ? scale_log2 / (ATTN_LOG2E * o.softcap) : 0.f;
  r.out = o.softcap * ATTN_LOG2E;
  return r;
}
__device__ __forceinline__ float scaled_score(const ScoreScale& r, float s) {
  return r.cap ? r.out * tanh_exp(s * r.in) : s * r.scale_log2;
}

}  // namespace fc
