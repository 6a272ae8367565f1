// Shared by the state-space kernels.
#pragma once
#include "common.cuh"

namespace kvb {

__device__ __forceinline__ float ss_silu(float x) { return x / (1.f + expf(-x)); }
// the same for results that are rounded to 16 bits
__device__ __forceinline__ float ss_silu_fast(float x) { return __fdividef(x, 1.f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float ss_silu_for(float x) { return sizeof(T) == 2 ? ss_silu_fast(x) : ss_silu(x); }
__device__ __forceinline__ float ss_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// exp(x) of a small negative number: what it lacks to 1 keeps its relative precision (a decay is taken to high powers)
__device__ __forceinline__ float ss_decay(float x) { return 1.f + expm1f(x); }

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
