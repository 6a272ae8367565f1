// What grouped attention sees and where its rows lie, shared by the prep, prompt and single-token kernels.
#pragma once
#include "common.cuh"
#include "kvb200_layers.h"

namespace kvb {

constexpr float ATTN_LOG2E = 1.4426950408889634f;

// Position hi sees the positions [seen_from(hi), hi] and, of the first `keep`, those up to its own.
__host__ __device__ __forceinline__ int seen_from(const kvb_attention& a, int hi) {
  if (a.chunk > 0) return hi / a.chunk * a.chunk;
  return a.window > 0 && hi >= a.window ? hi - a.window + 1 : 0;
}

// Row of a position: without a ring the position itself; with one the first `head` positions have rows of their own and the others
// share `ring` rows.
__host__ __device__ __forceinline__ int row_of(const kvb_attention& a, int pos) {
  return a.ring == 0 || pos < a.head ? pos : a.head + (pos - a.head) % a.ring;
}

__device__ __forceinline__ float attn_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float attn_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// tanh z = 1 - 2 / (1 + e^2z): absolute error of the order of 1e-7, which is what a soft cap wants (cap · tanh(score / cap) is a sum's exponent)
__device__ __forceinline__ float cap_tanh(float z) { return fmaf(-2.f, attn_rcp(1.f + attn_exp2(2.f * ATTN_LOG2E * z)), 1.f); }

// The same by the Taylor series up to z^9 for |z| <= 0.3 (what it leaves out is below 1e-7 of the result), two values at a time.
constexpr float CAP_SERIES = 0.3f;
__device__ __forceinline__ float2 cap_tanh_series(float2 z) {
  const float2 q = fmul2(z, z);
  float2 r = ffma2(q, make_float2(62.f / 2835.f, 62.f / 2835.f), make_float2(-17.f / 315.f, -17.f / 315.f));
  r = ffma2(q, r, make_float2(2.f / 15.f, 2.f / 15.f));
  r = ffma2(q, r, make_float2(-1.f / 3.f, -1.f / 3.f));
  return ffma2(fmul2(q, r), z, z);
}

}  // namespace kvb
