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

// Blocks that position hi sees (at most as many as there are rows for: padding may lie beyond the cache).
__host__ __device__ __forceinline__ int blocks_seen(const kvb_attention& a, int hi) {
  const int before = hi - a.window + 1;  // positions ahead of the window
  if (a.pool == 0 || before <= 0) return 0;
  const int n = before / a.pool;
  return n < a.head ? n : a.head;
}

// Row of a position: without a ring the position itself; with one the first `head` positions have rows of their own and the others
// share `ring` rows; with pooled blocks the first `head` rows are theirs.
__host__ __device__ __forceinline__ int row_of(const kvb_attention& a, int pos) {
  if (a.pool > 0) return a.head + pos % a.ring;
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

// Below CAP_SERIES tanh z = z (1 - z^2/3 + 2 z^4/15 - 17 z^6/315 + 62 z^8/2835), which leaves out less than 1e-7 of the result. A score that is
// capped that way is a polynomial in its square times the score: the coefficients take the factors on both sides.
constexpr float CAP_SERIES = 0.3f;
struct CapSeries {
  float c0, c1, c2, c3, c4;
  __host__ __device__ __forceinline__ CapSeries(float in, float out) {
    const float q = in * in;
    c0 = in * out;
    c1 = c0 * q * (-1.f / 3.f);
    c2 = c0 * q * q * (2.f / 15.f);
    c3 = c0 * q * q * q * (-17.f / 315.f);
    c4 = c0 * q * q * q * q * (62.f / 2835.f);
  }
  // with a last coefficient that has underflowed, minus infinity would not stay what it is
  __host__ __device__ __forceinline__ bool usable() const { return c4 > 1e-37f; }
};
// out · tanh(in · x) + add, two values at a time; minus infinity stays
__device__ __forceinline__ float2 cap_series(const CapSeries& s, float2 x, float2 add) {
  const float2 q = fmul2(x, x);
  float2 r = ffma2(q, make_float2(s.c4, s.c4), make_float2(s.c3, s.c3));
  r = ffma2(q, r, make_float2(s.c2, s.c2));
  r = ffma2(q, r, make_float2(s.c1, s.c1));
  r = ffma2(q, r, make_float2(s.c0, s.c0));
  return ffma2(x, r, add);
}

}  // namespace kvb
