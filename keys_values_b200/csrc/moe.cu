// Routed experts: softmax or sigmoid router with top-k choice, rows sorted by expert, grouped products.
//
//   route  one warp per token: scores from the fp32 router logits; the k largest, with a correction that only the choice sees and out of
//          the best groups of neighbouring experts, if the router has these; a rank within every chosen expert;
//   plan   one CTA: rows of an expert start at a multiple of the row tile; table of tiles for the grouped products;
//   gather rows of the chosen tokens into the sorted buffer;
//   gemm   out = act(W_e · in) per tile of rows of one expert; a gated unit has the rows of gate and up projection in turns, so
//          that silu(gate) · up is part of the product. bf16: tcgen05 with the expert's weight rows as the
//          M = 128 operand and the tokens as N (16 .. 256 columns), so that a decode step with a handful of tokens per
//          expert streams the weights without padding the token side to 128; fp32: CUDA cores.
// The weighted sum over a token's experts is part of the kernel that closes the layer (layer_edge.cu).
#include <cuda.h>

#include "common.cuh"
#include "kvb200_layers.h"

namespace kvb {

constexpr int ROUTE_WARPS = 8;
constexpr int ROUTE_TOKENS = 4;  // tokens of a warp, at most; a CTA counts its choices first and takes its rows of every expert at once
constexpr int ROUTE_MAX_EXPERTS = 2048;

__global__ void __launch_bounds__(ROUTE_WARPS * 32)
moe_route_kernel(const float* __restrict__ logits, int* __restrict__ expert, float* __restrict__ weight, int* __restrict__ row,
                 int* __restrict__ counters, long long n, int E, int top, int per_warp, const kvb_router r) {
  extern __shared__ float sc_all[];
  int* const local = reinterpret_cast<int*>(sc_all + ROUTE_WARPS * (E + r.groups));  // choices of this CTA per expert, then their first rows
  for (int e = threadIdx.x; e < E; e += ROUTE_WARPS * 32) local[e] = 0;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sc = sc_all + warp * (E + r.groups);  // choice scores; scores of the groups
  float* gs = sc + E;
  const long long tok0 = (long long)blockIdx.x * ROUTE_WARPS * per_warp;
  for (int i = 0; i < per_warp; ++i) {
    const long long tok = tok0 + i * ROUTE_WARPS + warp;
    if (tok >= n) break;
    const float* z = logits + tok * E;
    float m = 0.f, l = 1.f;  // softmax: score = exp(z - m) / l
    if (r.score == 0) {
      m = -INFINITY;
      for (int e = lane; e < E; e += 32) m = fmaxf(m, z[e]);
      m = warp_max(m);
      l = 0.f;
      for (int e = lane; e < E; e += 32) l += expf(z[e] - m);
      l = warp_sum(l);
    }
    auto score = [&](int e) { return r.score == 0 ? expf(z[e] - m) / l : 1.f / (1.f + expf(-z[e])); };
    for (int e = lane; e < E; e += 32) sc[e] = score(e) + (r.correction ? r.correction[e] : 0.f);
    __syncwarp();
    if (r.groups > 1) {
      const int size = E / r.groups;
      for (int g = lane; g < r.groups; g += 32) {  // sum of the two largest
        float a = -INFINITY, b = -INFINITY;
        for (int e = g * size; e < (g + 1) * size; ++e) {
          const float v = sc[e];
          b = fmaxf(b, fminf(a, v));
          a = fmaxf(a, v);
        }
        gs[g] = size > 1 ? a + b : a;
      }
      __syncwarp();
      for (int g = lane; g < r.groups; g += 32) {
        int ahead = 0;  // groups that come before this one; ties: lower index first
        for (int o = 0; o < r.groups; ++o) ahead += gs[o] > gs[g] || (gs[o] == gs[g] && o < g);
        if (ahead >= r.keep)
          for (int e = g * size; e < (g + 1) * size; ++e) sc[e] = -INFINITY;
      }
      __syncwarp();
    }
    float chosen = 0.f;
    for (int k = 0; k < top; ++k) {
      float best = -INFINITY;
      int bi = 0x7fffffff;
      for (int e = lane; e < E; e += 32) {
        const float v = sc[e];
        if (v > best) {  // those that cannot be chosen are at minus infinity
          best = v;
          bi = e;
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (ov > best || (ov == best && oi < bi)) {
          best = ov;
          bi = oi;
        }
      }
      if (bi >= E) bi = 0;  // scores that are not numbers: any expert
      const float w = score(bi);
      chosen += w;
      if (lane == 0) {
        expert[tok * top + k] = bi;
        weight[tok * top + k] = w;
        row[tok * top + k] = atomicAdd(&local[bi], 1);
        sc[bi] = -INFINITY;
      }
      __syncwarp();
    }
    if (r.renormalize)
      for (int k = lane; k < top; k += 32) weight[tok * top + k] = weight[tok * top + k] / (chosen + r.eps);
    __syncwarp();
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += ROUTE_WARPS * 32)
    if (local[e] > 0) local[e] = atomicAdd(&counters[e], local[e]);
  __syncthreads();
  for (int i = threadIdx.x; i < ROUTE_WARPS * per_warp * top; i += ROUTE_WARPS * 32) {
    const long long at = tok0 * top + i;
    if (at < n * top) row[at] += local[expert[at]];
  }
}

// Exclusive prefix over the experts' tile counts, tile table. One CTA of 1024 threads.
__global__ void __launch_bounds__(1024)
moe_plan_kernel(int* __restrict__ counters, int* __restrict__ plan, int* __restrict__ tile_expert, int* __restrict__ tile_row, int E,
                int tile, int max_tiles) {
  __shared__ int sums[32];
  __shared__ int carry;
  if (threadIdx.x == 0) carry = 0;
  __syncthreads();
  for (int e0 = 0; e0 < E; e0 += 1024) {
    const int e = e0 + threadIdx.x;
    const int nt = e < E ? (counters[e] + tile - 1) / tile : 0;
    int v = nt;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int t = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += t;
    }
    if (lane == 31) sums[warp] = v;
    __syncthreads();
    if (warp == 0) {
      int s = sums[lane];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int t = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += t;
      }
      sums[lane] = s;
    }
    __syncthreads();
    const int base = carry + (warp > 0 ? sums[warp - 1] : 0) + v - nt;
    if (e < E) {
      counters[e] = base * tile;  // first row of the expert
      for (int i = 0; i < nt && base + i < max_tiles; ++i) {
        tile_expert[base + i] = e;
        tile_row[base + i] = (base + i) * tile;
      }
    }
    __syncthreads();
    if (threadIdx.x == 1023) carry += sums[31];
    __syncthreads();
  }
  if (threadIdx.x == 0) plan[0] = min(carry, max_tiles);
}

__global__ void moe_rows_kernel(const int* __restrict__ expert, const int* __restrict__ counters, int* __restrict__ row, long long n) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) row[i] += counters[expert[i]];
}

template <typename T, int V>
__global__ void __launch_bounds__(128)
moe_gather_kernel(const T* __restrict__ h, const int* __restrict__ row, T* __restrict__ sorted, int top, int width, long long ld) {
  struct alignas(sizeof(T) * V) Vec { T v[V]; };
  const long long n = blockIdx.x;
  for (int c = threadIdx.x * V; c < ld; c += 128 * V) {
    Vec x;
    if (c < width) {
      x = *reinterpret_cast<const Vec*>(h + n * width + c);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) x.v[i] = from_f32<T>(0.f);
    }
    for (int k = 0; k < top; ++k) *reinterpret_cast<Vec*>(sorted + (long long)row[n * top + k] * ld + c) = x;
  }
}

// silu(gate) · up; for results that are rounded to 16 bits with the fast exponential and quotient
template <typename T> __device__ __forceinline__ float moe_glu(float gate, float up) {
  return sizeof(T) == 2 ? __fdividef(gate, 1.f + __expf(-gate)) * up : gate / (1.f + expf(-gate)) * up;
}

__device__ __forceinline__ float moe_act(float v, int act) {
  if (act == 1) {
    v = fmaxf(v, 0.f);
    return v * v;
  }
  return v;
}

// ---- CUDA-core product: 32 rows x 64 features per CTA. act 2: features 2 f and 2 f + 1 are gate and up of result f
constexpr int MS_R = 32, MS_F = 64, MS_K = 32;
template <typename T>
__global__ void __launch_bounds__(256)
moe_gemm_simple_kernel(const T* __restrict__ in, const T* __restrict__ w, T* __restrict__ out, const int* __restrict__ plan,
                       const int* __restrict__ tile_expert, const int* __restrict__ tile_row, int tile, int n_out, int k, long long ldk,
                       long long ldo, int act) {
  __shared__ float sa[MS_K][MS_R + 1];
  __shared__ float sw[MS_K][MS_F + 1];
  const int sub = tile / MS_R;
  const int ti = blockIdx.x / sub;
  if (ti >= plan[0]) return;
  const long long r0 = (long long)tile_row[ti] + (blockIdx.x % sub) * MS_R;
  const long long e = tile_expert[ti];
  const int f0 = blockIdx.y * MS_F;
  const T* we = w + e * n_out * ldk;
  const int tr = threadIdx.x / 32, tf = threadIdx.x % 32;  // rows tr + 8 i, features 2 tf and 2 tf + 1
  float acc[4][2] = {};
  for (int k0 = 0; k0 < k; k0 += MS_K) {
    for (int i = threadIdx.x; i < MS_R * MS_K; i += 256) {
      const int r = i / MS_K, kk = i % MS_K;
      sa[kk][r] = k0 + kk < k ? to_f32(in[(r0 + r) * ldk + k0 + kk]) : 0.f;
    }
    for (int i = threadIdx.x; i < MS_F * MS_K; i += 256) {
      const int f = i / MS_K, kk = i % MS_K;
      sw[kk][f] = (f0 + f < n_out && k0 + kk < k) ? to_f32(we[(long long)(f0 + f) * ldk + k0 + kk]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int kk = 0; kk < MS_K; ++kk) {
      const float w0 = sw[kk][2 * tf], w1 = sw[kk][2 * tf + 1];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float a = sa[kk][tr + 8 * i];
        acc[i][0] = fmaf(a, w0, acc[i][0]);
        acc[i][1] = fmaf(a, w1, acc[i][1]);
      }
    }
    __syncthreads();
  }
  if (act == 2) {
    const int f = f0 / 2 + tf;
    if (f < ldo) {
#pragma unroll
      for (int i = 0; i < 4; ++i) out[(r0 + tr + 8 * i) * ldo + f] = from_f32<T>(2 * f < n_out ? moe_glu<T>(acc[i][0], acc[i][1]) : 0.f);
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int f = f0 + 2 * tf + j;
      if (f < ldo) out[(r0 + tr + 8 * i) * ldo + f] = from_f32<T>(f < n_out ? moe_act(acc[i][j], act) : 0.f);
    }
}

// out[n, c] = silu(x[n, c]) · x[n, up + c], zero in the columns from ff to ldo. A CTA has one row.
// what a gated feed-forward does with gate and up projection
struct SiluUnit {
  template <typename T> __device__ __forceinline__ float of(float g, float u) const { return moe_glu<T>(g, u); }
};
// g · sigmoid(1.702 g) · (u + 1) with g at most the limit and u within it on both sides
struct ClampedUnit {
  float limit;
  template <typename T> __device__ __forceinline__ float of(float g, float u) const {
    g = fminf(g, limit);
    const float e = -1.702f * g;
    const float s = sizeof(T) == 2 ? __fdividef(g, 1.f + __expf(e)) : g / (1.f + expf(e));
    return s * (fminf(fmaxf(u, -limit), limit) + 1.f);
  }
};

template <typename T, int V, typename Unit>
__global__ void __launch_bounds__(256)
glu_kernel(const T* __restrict__ x, T* __restrict__ out, long long ldx, int up, int ff, int ldo, const Unit unit) {
  struct alignas(sizeof(T) * V) Vec { T v[V]; };
  x += blockIdx.x * ldx;
  out += (long long)blockIdx.x * ldo;
#pragma unroll 4
  for (int c = threadIdx.x * V; c < ldo; c += blockDim.x * V) {
    Vec y;
    if (c < ff) {
      const Vec g = *reinterpret_cast<const Vec*>(x + c), u = *reinterpret_cast<const Vec*>(x + up + c);
#pragma unroll
      for (int e = 0; e < V; ++e) y.v[e] = from_f32<T>(unit.template of<T>(to_f32(g.v[e]), to_f32(u.v[e])));
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) y.v[e] = from_f32<T>(0.f);
    }
    *reinterpret_cast<Vec*>(out + c) = y;
  }
}

template <typename T, typename Unit>
static int glu_launch(const void* x, void* out, long long n, long long ldx, int up, int ff, int ldo, const Unit& unit, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = ff % V == 0 && up % V == 0 && ldx % V == 0 && ldo % V == 0;
  int threads = ((vec ? ldo / V : ldo) + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  if (vec) glu_kernel<T, V><<<(unsigned)n, threads, 0, s>>>((const T*)x, (T*)out, ldx, up, ff, ldo, unit);
  else glu_kernel<T, 1><<<(unsigned)n, threads, 0, s>>>((const T*)x, (T*)out, ldx, up, ff, ldo, unit);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <typename T>
static int glu_type(const void* x, void* out, long long n, long long ldx, int up, int ff, int ldo, float limit, cudaStream_t s) {
  return limit > 0.f ? glu_launch<T>(x, out, n, ldx, up, ff, ldo, ClampedUnit{limit}, s) : glu_launch<T>(x, out, n, ldx, up, ff, ldo, SiluUnit{}, s);
}

int moe_gemm_tc(const void* in, const void* w, void* out, const int* plan, const int* tile_expert, const int* tile_row, int tile,
                int max_tiles, int n_expert, int n_out, int k, long long ldk, long long ldo, int act, int* status, cudaStream_t s);

}  // namespace kvb

extern "C" int kvb_moe_route(const float* logits, int* expert, float* weight, int* row, int* counters, int* plan, int* tile_expert,
                             int* tile_row, long long n, int n_expert, int top, int tile, int max_tiles, const kvb_router* router, void* stream) {
  using namespace kvb;
  if (n <= 0 || n_expert <= 0 || top <= 0 || top > n_expert || tile <= 0 || !router) return KVB_ERR_ARG;
  const kvb_router r = *router;
  if (r.groups < 1 || n_expert % r.groups || r.keep < 1 || r.keep > r.groups || r.keep * (n_expert / r.groups) < top || r.score < 0 || r.score > 1)
    return KVB_ERR_ARG;
  if (n_expert > ROUTE_MAX_EXPERTS) return KVB_ERR_TOO_LARGE;
  cudaStream_t s = (cudaStream_t)stream;
  if (cudaMemsetAsync(counters, 0, sizeof(int) * n_expert, s) != cudaSuccess) return KVB_ERR_CUDA;
  const int per_warp = n >= 148LL * 8 * ROUTE_WARPS * ROUTE_TOKENS / 4 ? ROUTE_TOKENS : 1;
  const int tokens = ROUTE_WARPS * per_warp;
  const size_t smem = (size_t)ROUTE_WARPS * (n_expert + r.groups) * sizeof(float) + (size_t)n_expert * sizeof(int);
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
  moe_route_kernel<<<(unsigned)((n + tokens - 1) / tokens), ROUTE_WARPS * 32, smem, s>>>(logits, expert, weight, row, counters, n, n_expert, top,
                                                                                       per_warp, r);
  moe_plan_kernel<<<1, 1024, 0, s>>>(counters, plan, tile_expert, tile_row, n_expert, tile, max_tiles);
  const long long m = n * top;
  moe_rows_kernel<<<(unsigned)((m + 255) / 256), 256, 0, s>>>(expert, counters, row, m);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_moe_gather(const void* h, const int* row, void* sorted, long long n, int top, int width, long long ld, int dtype,
                              void* stream) {
  using namespace kvb;
  if (n <= 0 || top <= 0 || ld < width) return KVB_ERR_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  const unsigned g = (unsigned)n;
  const bool vec = width % 8 == 0 && ld % 8 == 0;
  if (dtype == 0) {
    if (vec) moe_gather_kernel<float, 4><<<g, 128, 0, s>>>((const float*)h, row, (float*)sorted, top, width, ld);
    else moe_gather_kernel<float, 1><<<g, 128, 0, s>>>((const float*)h, row, (float*)sorted, top, width, ld);
  } else if (dtype == 1) {
    if (vec) moe_gather_kernel<__nv_bfloat16, 8><<<g, 128, 0, s>>>((const __nv_bfloat16*)h, row, (__nv_bfloat16*)sorted, top, width, ld);
    else moe_gather_kernel<__nv_bfloat16, 1><<<g, 128, 0, s>>>((const __nv_bfloat16*)h, row, (__nv_bfloat16*)sorted, top, width, ld);
  } else {
    return KVB_ERR_ARG;
  }
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_moe_gemm(const void* in, const void* w, void* out, const int* plan, const int* tile_expert, const int* tile_row,
                            int tile, int max_tiles, int n_expert, int n_out, int k, long long ldk, long long ldo, int act, int dtype,
                            int simple, int* status, void* stream) {
  using namespace kvb;
  if (max_tiles <= 0 || n_out <= 0 || k <= 0 || ldk < k || ldo < (act == 2 ? n_out / 2 : n_out) || tile <= 0 || (act == 2 && n_out % 2))
    return KVB_ERR_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == 1 && !simple)
    return moe_gemm_tc(in, w, out, plan, tile_expert, tile_row, tile, max_tiles, n_expert, n_out, k, ldk, ldo, act, status, s);
  if (tile % MS_R) return KVB_ERR_ARG;
  const long long features = act == 2 ? 2 * ldo : ldo;
  const dim3 grid(max_tiles * (tile / MS_R), (unsigned)((features + MS_F - 1) / MS_F));
  if (dtype == 0)
    moe_gemm_simple_kernel<float><<<grid, 256, 0, s>>>((const float*)in, (const float*)w, (float*)out, plan, tile_expert, tile_row, tile,
                                                       n_out, k, ldk, ldo, act);
  else if (dtype == 1)
    moe_gemm_simple_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>((const __nv_bfloat16*)in, (const __nv_bfloat16*)w, (__nv_bfloat16*)out,
                                                               plan, tile_expert, tile_row, tile, n_out, k, ldk, ldo, act);
  else return KVB_ERR_ARG;
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_glu(const void* x, void* out, long long n, long long ldx, int up, int ff, int ldo, float limit, int dtype, void* stream) {
  if (n <= 0 || ff <= 0 || up < ff || ldx < up + ff || ldo < ff || n > 0x7fffffffLL) return KVB_ERR_ARG;
  if (dtype == 0) return kvb::glu_type<float>(x, out, n, ldx, up, ff, ldo, limit, (cudaStream_t)stream);
  if (dtype == 1) return kvb::glu_type<__nv_bfloat16>(x, out, n, ldx, up, ff, ldo, limit, (cudaStream_t)stream);
  return KVB_ERR_ARG;
}
