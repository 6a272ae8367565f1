// Shared by the state-space kernels.
#pragma once
#include "common.cuh"
#include "kvb200_layers.h"

namespace kvb {

__device__ __forceinline__ float ss_silu(float x) { return x / (1.f + expf(-x)); }
// the same for results that are rounded to 16 bits
__device__ __forceinline__ float ss_silu_fast(float x) { return __fdividef(x, 1.f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float ss_silu_for(float x) { return sizeof(T) == 2 ? ss_silu_fast(x) : ss_silu(x); }
__device__ __forceinline__ float ss_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// log(1 + exp(x)) = max(x, 0) + log(1 + e) with e = exp(−|x|) <= 1, and log(1 + e) = 2 artanh(s), s = e / (2 + e) <= 1/3: seven terms of
// the series leave a relative error of 2e-8
__device__ __forceinline__ float ss_softplus_fast(float x) {
  const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), q = s * s;
  float r = fmaf(q, 1.f / 13.f, 1.f / 11.f);
  r = fmaf(q, r, 1.f / 9.f);
  r = fmaf(q, r, 1.f / 7.f);
  r = fmaf(q, r, 1.f / 5.f);
  r = fmaf(q, r, 1.f / 3.f);
  r = fmaf(q, r, 1.f);
  return fmaf(2.f * s, r, fmaxf(x, 0.f));
}

// exp(x) of a small negative number: what it lacks to 1 keeps its relative precision (a decay is taken to high powers)
__device__ __forceinline__ float ss_decay(float x) { return 1.f + expm1f(x); }

// logarithm of the decay of key channel c of a gated linear attention, from the token's low-rank input a
__device__ __forceinline__ float gl_log_decay(const kvb_gated_linear& g, const float* a, int c) {
  float z = g.bias[c];
#pragma unroll 8
  for (int r = 0; r < g.rank; ++r) z = fmaf(a[r], g.w[(long long)r * g.heads * g.np + c], z);
  return -ss_softplus(-z) * g.inv_tau;
}

// The recurrence S_t = a_t S_(t-1) + dt_t B_t x_t^T, y_t = S_t^T C_t + skip x_t, with a_t = exp(-exp(a_log) dt_t) and dt_t from the joint
// projection, or (decay not NULL) with a fixed decay per head and step 1, without skip.
struct ScanParams {
  const float *dt_bias, *a_log, *skip;  // (heads)
  const float* decay;                   // (heads): the decay, in the chunked kernel its log2; NULL: from step sizes
  const int *slots, *start, *count;
  float* state;                         // (slots, heads, np, vdp)
  long long ld;                         // of the joint projection, whose step sizes start at column dt_col
  int T, dt_col, heads, groups, vdp, np, inner, channels;
};

}  // namespace kvb
