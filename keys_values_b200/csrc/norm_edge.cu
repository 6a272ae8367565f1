// What happens between two sublayers of a model whose layers have norms before and / or after each sublayer, in one pass over
// the fp32 residual stream: weighted sum of a token's routed experts, norm of the sublayer's output, residual sum, what a loop adds
// ahead of a pass (embedding row of the token, a vector), norm for the next sublayer (or the stream itself, where sublayers read
// that). Also the entry into the stack (embedding rows only) and the norm of rows in front of the output head.
//
// A CTA has one row, which stays in registers; means and squared deviations are separate sums (no cancellation).
//
// What a sublayer reads may pass a short causal convolution over time. A single token finds the inputs before it in a ring of its sequence and
// is done here; several tokens pass the convolution of ssm.cu afterwards.
#include <type_traits>

#include "common.cuh"
#include "kvb200_layers.h"

namespace kvb {

struct NormEdgeParams {
  const float* x_in;
  const void* sub;
  const float* after;
  float* x_out;
  const float* before;
  void* h;
  const long long* idx;
  const void* embed;
  long long vocab;
  const float* step;
  const void* expert_out;
  const int* expert_row;
  const float* expert_w;
  long long expert_ld;
  int top;
  int width;
  float eps, inv_width;
  int* status;
  kvb_edge_tokens tok;
};

template <typename T, int V> struct RowVec {
  static __device__ __forceinline__ void load(const T* p, float (&v)[V]) {
    if constexpr (V == 1) {
      v[0] = to_f32(*p);
    } else if constexpr (sizeof(T) == 4) {
      const float4 t = *reinterpret_cast<const float4*>(p);
      v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    } else {
      const uint2 t = *reinterpret_cast<const uint2*>(p);
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
      v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    }
  }
  static __device__ __forceinline__ void store(T* p, const float (&v)[V]) {
    if constexpr (V == 1) {
      *p = from_f32<T>(v[0]);
    } else if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
      *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
    }
  }
};

// row of the position table for row n of the pass; padding may lie beyond the table
__device__ __forceinline__ long long table_row(const NormEdgeParams& p, long long n) {
  const long long pos = p.tok.start[n / p.tok.T] + n % p.tok.T;
  return pos < p.tok.table_rows ? pos : p.tok.table_rows - 1;
}

// columns [c, c + V) of h of a single token pass the convolution; the ring takes h (its row is none of those that are read)
template <typename T, int V>
__device__ __forceinline__ void conv_single(const NormEdgeParams& p, int b, int c, float (&h)[V]) {
  const int taps = p.tok.taps, pos = p.tok.start[b];
  T* ring = static_cast<T*>(p.tok.conv_ring) + (long long)p.tok.slots[b] * taps * p.width + c;
  float w[V], v[V], s[V];
  RowVec<float, V>::load(p.tok.conv_w + (long long)(taps - 1) * p.width + c, w);
#pragma unroll
  for (int e = 0; e < V; ++e) s[e] = w[e] * to_f32(from_f32<T>(h[e]));  // as the convolution of several tokens reads it
#pragma unroll 4
  for (int k = 1; k < taps; ++k) {
    if (k > pos) break;
    RowVec<float, V>::load(p.tok.conv_w + (long long)(taps - 1 - k) * p.width + c, w);
    RowVec<T, V>::load(ring + (long long)((pos - k) % taps) * p.width, v);
#pragma unroll
    for (int e = 0; e < V; ++e) s[e] = fmaf(w[e], v[e], s[e]);
  }
  if (p.tok.count[b] > 0) RowVec<T, V>::store(ring + (long long)(pos % taps) * p.width, h);
#pragma unroll
  for (int e = 0; e < V; ++e) h[e] = s[e];
}

// sum over the CTA; every call of a row has its own `red`
template <int TH>
__device__ __forceinline__ float row_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < TH / 32; ++i) s += red[i];
  return s;
}

// y = norm(x) without the weight; entries beyond the row must be zero and stay zero
template <int TH, int NC, int V, bool CENTER>
__device__ __forceinline__ float row_norm_factor(float (&x)[NC][V], const NormEdgeParams& p, float (*red)[TH / 32]) {
  if (CENTER) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) s += x[i][e];
    const float mean = row_sum<TH>(s, red[0]) * p.inv_width;
#pragma unroll
    for (int i = 0; i < NC; ++i)
      if ((i * TH + (int)threadIdx.x) * V < p.width) {
#pragma unroll
        for (int e = 0; e < V; ++e) x[i][e] -= mean;
      }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NC; ++i)
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(x[i][e], x[i][e], ss);
  return 1.f / sqrtf(row_sum<TH>(ss, red[1]) * p.inv_width + p.eps);
}

template <typename T, int V, int TH, int NC, bool CENTER, bool EXPERTS>
__global__ void __launch_bounds__(TH)
norm_edge_kernel(const NormEdgeParams p) {
  __shared__ float red[4][TH / 32];
  const long long n = blockIdx.x, o = n * p.width;
  float x[NC][V], y[NC][V];
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = (i * TH + threadIdx.x) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) x[i][e] = y[i][e] = 0.f;
    if (c >= p.width) continue;
    if (p.sub) RowVec<T, V>::load(static_cast<const T*>(p.sub) + o + c, y[i]);
    if (p.x_in) RowVec<float, V>::load(p.x_in + o + c, x[i]);
  }
  // up to four experts at a time, so that their rows are on their way together
  for (int k0 = 0; EXPERTS && k0 < p.top; k0 += 4) {
    const T* src[4];
    float w[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const bool in = k0 + k < p.top;
      src[k] = static_cast<const T*>(p.expert_out) + (long long)p.expert_row[n * p.top + (in ? k0 + k : k0)] * p.expert_ld;
      w[k] = in ? p.expert_w[n * p.top + k0 + k] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = (i * TH + threadIdx.x) * V;
      if (c >= p.width) continue;
      float e[4][V];
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (k0 + k < p.top) RowVec<T, V>::load(src[k] + c, e[k]);
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (k0 + k < p.top) {
#pragma unroll
          for (int j = 0; j < V; ++j) y[i][j] = fmaf(w[k], e[k][j], y[i][j]);
        }
    }
  }
  long long tok = 0;
  if (p.embed) {
    tok = p.idx[n];
    if (tok < 0 || tok >= p.vocab) {
      if (p.status) atomicCAS(p.status, 0, STATUS_BAD_INDEX);
      tok = 0;
    }
  }
  float r = 1.f;
  if (p.after) r = row_norm_factor<TH, NC, V, CENTER>(y, p, red);
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = (i * TH + threadIdx.x) * V;
    if (c >= p.width) continue;
    float w[V];
    if (p.after) {
      RowVec<float, V>::load(p.after + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = fmaf(y[i][e] * r, w[e], x[i][e]);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] += y[i][e];
    }
    if (p.embed) {
      RowVec<T, V>::load(static_cast<const T*>(p.embed) + tok * p.width + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] += w[e];
    }
    if (p.tok.table) {
      RowVec<T, V>::load(static_cast<const T*>(p.tok.table) + table_row(p, n) * p.width + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] += w[e];
    }
    if (p.step) {
      RowVec<float, V>::load(p.step + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] += w[e];
    }
    if (p.x_out) RowVec<float, V>::store(p.x_out + o + c, x[i]);
  }
  if (!p.h) return;
  if (p.before) r = row_norm_factor<TH, NC, V, CENTER>(x, p, red + 2);
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = (i * TH + threadIdx.x) * V;
    if (c >= p.width) continue;
    if (p.before) {
      float w[V];
      RowVec<float, V>::load(p.before + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = w[e] * (x[i][e] * r);
    }
    if (p.tok.conv_w) conv_single<T, V>(p, (int)n, c, x[i]);
    RowVec<T, V>::store(static_cast<T*>(p.h) + o + c, x[i]);
  }
}

template <typename T, int V, bool CENTER, bool EXPERTS>
static int norm_edge_launch(const NormEdgeParams& p, long long n, cudaStream_t s) {
  const unsigned g = (unsigned)n;
  if (n <= 148 && p.width > 128 * V) {  // few rows: latency counts, every thread has one access
    if (p.width <= 256 * V) norm_edge_kernel<T, V, 256, 1, CENTER, EXPERTS><<<g, 256, 0, s>>>(p);
    else if (p.width <= 512 * V) norm_edge_kernel<T, V, 512, 1, CENTER, EXPERTS><<<g, 512, 0, s>>>(p);
    else if (p.width <= 1024 * V) norm_edge_kernel<T, V, 1024, 1, CENTER, EXPERTS><<<g, 1024, 0, s>>>(p);
    else if (p.width <= 8192 * V) norm_edge_kernel<T, V, 1024, 8, CENTER, EXPERTS><<<g, 1024, 0, s>>>(p);
    else return KVB_ERR_TOO_LARGE;
  } else if (p.width <= 128 * V) norm_edge_kernel<T, V, 128, 1, CENTER, EXPERTS><<<g, 128, 0, s>>>(p);
  else if (p.width <= 256 * V) norm_edge_kernel<T, V, 128, 2, CENTER, EXPERTS><<<g, 128, 0, s>>>(p);
  else if (p.width <= 512 * V) norm_edge_kernel<T, V, 128, 4, CENTER, EXPERTS><<<g, 128, 0, s>>>(p);
  else if (p.width <= 1024 * V) norm_edge_kernel<T, V, 256, 4, CENTER, EXPERTS><<<g, 256, 0, s>>>(p);
  else if (p.width <= 2048 * V) norm_edge_kernel<T, V, 512, 4, CENTER, EXPERTS><<<g, 512, 0, s>>>(p);
  else if (p.width <= 8192 * V) norm_edge_kernel<T, V, 1024, 8, CENTER, EXPERTS><<<g, 1024, 0, s>>>(p);
  else return KVB_ERR_TOO_LARGE;
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <typename T>
static int norm_edge_type(const NormEdgeParams& p, long long n, int center, cudaStream_t s) {
  auto launch = [&](auto vec, auto experts) {
    constexpr int V = decltype(vec)::value;
    constexpr bool E = decltype(experts)::value;
    return center ? norm_edge_launch<T, V, true, E>(p, n, s) : norm_edge_launch<T, V, false, E>(p, n, s);
  };
  using One = std::integral_constant<int, 1>;
  using Four = std::integral_constant<int, 4>;
  if (p.top > 0) return p.width % 4 == 0 ? launch(Four{}, std::true_type{}) : launch(One{}, std::true_type{});
  return p.width % 4 == 0 ? launch(Four{}, std::false_type{}) : launch(One{}, std::false_type{});
}

}  // namespace kvb

extern "C" int kvb_norm_edge(const float* x_in, const void* sub, const void* expert_out, const int* expert_row, const float* expert_w, int top,
                             long long expert_ld, const float* after, float* x_out, const float* before, void* h, const long long* idx,
                             const void* embed, long long vocab, const float* step, long long n, int width, float eps, int center,
                             int dtype, const kvb_edge_tokens* tokens, int* status, void* stream) {
  if (tokens && (tokens->T <= 0 || n % tokens->T || n / tokens->T > 65535 || !tokens->slots || !tokens->start || !tokens->count ||
                 (tokens->table && tokens->table_rows <= 0) ||
                 (tokens->conv_w && (!tokens->conv_ring || tokens->taps <= 0 || !h || tokens->T > 1))))
    return KVB_ERR_ARG;
  if (n <= 0 || n > 0x7fffffffLL || width <= 0 || (before && !h) || (embed && !idx) || (after && !sub && !expert_out) ||
      (expert_out && (!expert_row || !expert_w || top <= 0 || expert_ld < width)))
    return KVB_ERR_ARG;
  if (expert_out && width % 4 == 0 && expert_ld % 4) return KVB_ERR_ALIGN;
  kvb::NormEdgeParams p;
  p.x_in = x_in; p.sub = sub; p.after = after; p.x_out = x_out; p.before = before; p.h = h; p.idx = idx; p.embed = embed;
  p.vocab = vocab; p.step = step; p.width = width; p.eps = eps; p.inv_width = 1.f / (float)width; p.status = status;
  p.expert_out = expert_out; p.expert_row = expert_row; p.expert_w = expert_w; p.expert_ld = expert_ld; p.top = expert_out ? top : 0;
  p.tok = tokens ? *tokens : kvb_edge_tokens{};
  if (dtype == 0) return kvb::norm_edge_type<float>(p, n, center, (cudaStream_t)stream);
  if (dtype == 1) return kvb::norm_edge_type<__nv_bfloat16>(p, n, center, (cudaStream_t)stream);
  return KVB_ERR_ARG;
}
