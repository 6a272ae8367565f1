// What happens between two layers of a model with fp32 residual stream, in one pass over the data: residual sum of
// the parallel sublayers (mixer and weighted expert outputs), average over the depth history, RMS norm with one
// gain, token shift. The first layer's variant takes its rows from the token and bigram embeddings.
//
// One CTA walks over a few consecutive tokens of a row and keeps the previous token's normed row in registers of the
// threads that own its columns; the token before its first one is recomputed (or, at the start of a pass, read from the
// sequence's state), so the pass needs no second kernel for the shift. The arithmetic of a token is the same whichever CTA
// computes it: prompts and single-token steps agree bit for bit given equal inputs.
#include "common.cuh"
#include "kvb200_layers.h"

namespace kvb {

constexpr int EDGE_THREADS = 256;  // of the plain norm; the layer edge takes 256 or 512 by width

struct EdgeParams {
  // embedding source
  const long long* idx;
  const int* prev_token;
  const void *embed, *bigram;
  long long buckets, mul_prev, mul_cur, vocab;
  int* status;
  // residual source
  const float* x_in;
  const void* mix;
  const void* expert_out;
  const int* expert_row;
  const float* expert_w;
  int top;
  long long expert_ld;
  // depth history
  float* hist;
  int n_hist;
  long long hist_stride;
  const float* coef;
  float* x_out;
  // norm and shift
  const float *gain, *shift;
  float* state;
  void *h, *hs;
  const int *slots, *start, *count;
  int B, T, width, run;
  float eps;
};

template <typename T, int V> struct EdgeVec;
template <> struct EdgeVec<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct EdgeVec<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  }
};
template <typename T> struct EdgeVec<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f32(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_f32<T>(v[0]); }
};

// Sum over the CTA of TH threads; `red` has one float per warp, alternating between two buffers so that one barrier is enough.
template <int TH>
__device__ __forceinline__ float edge_block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < TH / 32; ++i) s += red[i];
  return s;
}

// token id n, reported and replaced by 0 if it is not in the vocabulary
__device__ __forceinline__ long long edge_token(const EdgeParams& p, long long n) {
  const long long tok = p.idx[n];
  if (tok >= 0 && tok < p.vocab) return tok;
  if (p.status) atomicCAS(p.status, 0, STATUS_BAD_INDEX);
  return 0;
}

// row of the bigram table for token t of row b
__device__ __forceinline__ long long edge_bigram_row(const EdgeParams& p, int b, int t) {
  const long long cur = edge_token(p, (long long)b * p.T + t);
  long long prev;
  if (t > 0) prev = edge_token(p, (long long)b * p.T + t - 1);
  else if (p.start[b] > 0) prev = p.prev_token[p.slots[b]];
  else return p.buckets;
  return (prev * p.mul_prev + cur * p.mul_cur) % p.buckets;
}

// x of token t for this thread's columns; `keep`: write the history and the stream. All loads of a token are issued before the
// first store, those of several streams together.
template <typename T, int V, int TH, int NC, bool EMBED>
__device__ __forceinline__ void edge_load(const EdgeParams& p, int b, int t, bool keep, float (&x)[NC][V]) {
  const long long n = (long long)b * p.T + t;
  const int c0 = threadIdx.x * V;
  constexpr int STEP = TH * V;
  if (EMBED) {
    const T* e = static_cast<const T*>(p.embed) + edge_token(p, n) * p.width;
    const T* g = p.bigram ? static_cast<const T*>(p.bigram) + edge_bigram_row(p, b, t) * p.width : nullptr;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = c0 + i * STEP;
      if (c >= p.width) continue;
      EdgeVec<T, V>::load(e + c, x[i]);
      if (g) {
        float y[V];
        EdgeVec<T, V>::load(g + c, y);
#pragma unroll
        for (int u = 0; u < V; ++u) x[i][u] += y[u];
      }
    }
    if (keep) {
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (c0 + i * STEP < p.width) EdgeVec<float, V>::store(p.hist + n * p.width + c0 + i * STEP, x[i]);
    }
    return;
  }
  constexpr int EARLY = 8;  // experts whose rows are looked up first
  int er[EARLY];
  float ew[EARLY];
  const int early = p.expert_out ? min(p.top, EARLY) : 0;
#pragma unroll
  for (int k = 0; k < EARLY; ++k) {
    er[k] = k < early ? p.expert_row[n * p.top + k] : 0;
    ew[k] = k < early ? p.expert_w[n * p.top + k] : 0.f;
  }
  const long long o = n * p.width;
  float fresh[NC][V], sub[NC][V];
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = c0 + i * STEP;
#pragma unroll
    for (int u = 0; u < V; ++u) x[i][u] = fresh[i][u] = sub[i][u] = 0.f;
    if (c >= p.width) continue;
    EdgeVec<float, V>::load(p.x_in + o + c, fresh[i]);
    EdgeVec<T, V>::load(static_cast<const T*>(p.mix) + o + c, sub[i]);
  }
  if (p.coef) {
#pragma unroll 4
    for (int j = 0; j < p.n_hist; ++j) {
      const float w = p.coef[j];
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int c = c0 + i * STEP;
        if (c >= p.width) continue;
        float y[V];
        EdgeVec<float, V>::load(p.hist + j * p.hist_stride + o + c, y);
#pragma unroll
        for (int u = 0; u < V; ++u) x[i][u] = fmaf(w, y[u], x[i][u]);
      }
    }
  }
  auto add_expert = [&](int row, float w) {
    const T* y0 = static_cast<const T*>(p.expert_out) + (long long)row * p.expert_ld;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = c0 + i * STEP;
      if (c >= p.width) continue;
      float y[V];
      EdgeVec<T, V>::load(y0 + c, y);
#pragma unroll
      for (int u = 0; u < V; ++u) sub[i][u] = fmaf(w, y[u], sub[i][u]);
    }
  };
#pragma unroll
  for (int k = 0; k < EARLY; ++k)
    if (k < early) add_expert(er[k], ew[k]);
  if (p.expert_out)
    for (int k = EARLY; k < p.top; ++k) add_expert(p.expert_row[n * p.top + k], p.expert_w[n * p.top + k]);
  const float w_new = p.coef ? p.coef[p.n_hist] : 1.f;
#pragma unroll
  for (int i = 0; i < NC; ++i)
#pragma unroll
    for (int u = 0; u < V; ++u) {
      fresh[i][u] += sub[i][u];
      x[i][u] = fmaf(w_new, fresh[i][u], x[i][u]);
    }
  if (keep) {
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = c0 + i * STEP;
      if (c >= p.width) continue;
      if (p.coef) EdgeVec<float, V>::store(p.hist + p.n_hist * p.hist_stride + o + c, fresh[i]);
      EdgeVec<float, V>::store(p.x_out + o + c, x[i]);
    }
  }
}

// TH threads with NC groups of V columns each
template <typename T, int V, int TH, int NC, bool EMBED>
__global__ void __launch_bounds__(TH)
layer_edge_kernel(const EdgeParams p) {
  __shared__ float red[2][TH / 32];
  const int b = blockIdx.y;
  const int t0 = blockIdx.x * p.run;
  const int t1 = min(t0 + p.run, p.T);
  const int first = (t0 > 0 && p.gain && p.shift) ? t0 - 1 : t0;
  float hp[NC][V];
  const bool shifted = p.gain && p.shift;
  if (shifted && t0 == 0) {
    const bool has = p.start[b] > 0;
    const float* st = p.state + (long long)p.slots[b] * p.width;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = (i * TH + threadIdx.x) * V;
#pragma unroll
      for (int e = 0; e < V; ++e) hp[i][e] = 0.f;
      if (has && c < p.width) EdgeVec<float, V>::load(st + c, hp[i]);
    }
  }
  const float gain = p.gain ? *p.gain : 0.f;
  for (int t = first; t < t1; ++t) {
    const bool keep = t >= t0;
    float x[NC][V];
    float ss = 0.f;
    edge_load<T, V, TH, NC, EMBED>(p, b, t, keep, x);
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = (i * TH + threadIdx.x) * V;
      if (c < p.width) {
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(x[i][e], x[i][e], ss);
      }
    }
    if (!p.gain) continue;
    ss = edge_block_sum<TH>(ss, red[t & 1]);
    const float r = gain / sqrtf(ss / (float)p.width + p.eps);
    const long long o = ((long long)b * p.T + t) * p.width;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = (i * TH + threadIdx.x) * V;
      if (c >= p.width) continue;
      float h[V];
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] = x[i][e] * r;
      if (keep) EdgeVec<T, V>::store(static_cast<T*>(p.h) + o + c, h);
      if (shifted) {
        if (keep) {
          float s[V], y[V];
          EdgeVec<float, V>::load(p.shift + c, s);
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] = fmaf(hp[i][e] - h[e], s[e], h[e]);
          EdgeVec<T, V>::store(static_cast<T*>(p.hs) + o + c, y);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) hp[i][e] = h[e];
      }
    }
  }
  // a single-token pass: this CTA was the only reader of the state of its sequence
  if (shifted && p.T == 1 && p.count[b] > 0) {
    float* st = p.state + (long long)p.slots[b] * p.width;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = (i * TH + threadIdx.x) * V;
      if (c < p.width) EdgeVec<float, V>::store(st + c, hp[i]);
    }
  }
}

// Passes of several tokens: the state is written after every CTA has read the old one. x: the stream the norm was taken of.
template <int V, int TH, int NC>
__global__ void __launch_bounds__(TH)
shift_state_kernel(const float* __restrict__ x, const float* __restrict__ gain_p, float* __restrict__ state, const int* __restrict__ slots,
                   const int* __restrict__ count, int T, int width, float eps) {
  __shared__ float red[TH / 32];
  const int b = blockIdx.x;
  if (count[b] <= 0) return;
  const float* xr = x + ((long long)b * T + count[b] - 1) * width;
  float v[NC][V];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = (i * TH + threadIdx.x) * V;
    if (c < width) {
      EdgeVec<float, V>::load(xr + c, v[i]);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[i][e], v[i][e], ss);
    }
  }
  ss = edge_block_sum<TH>(ss, red);
  const float r = *gain_p / sqrtf(ss / (float)width + eps);
  float* st = state + (long long)slots[b] * width;
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = (i * TH + threadIdx.x) * V;
    if (c < width) {
#pragma unroll
      for (int e = 0; e < V; ++e) v[i][e] *= r;
      EdgeVec<float, V>::store(st + c, v[i]);
    }
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(EDGE_THREADS)
scalar_rmsnorm_kernel(const float* __restrict__ x, const long long* __restrict__ rows, const float* __restrict__ gain_p, T* __restrict__ y,
                      int width, float eps) {
  __shared__ float red[EDGE_THREADS / 32];
  const long long n = blockIdx.x;
  const float* xr = x + (rows ? rows[n] : n) * width;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < width; c += EDGE_THREADS * V) {
    float v[V];
    EdgeVec<float, V>::load(xr + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
  }
  ss = edge_block_sum<EDGE_THREADS>(ss, red);
  const float r = *gain_p / sqrtf(ss / (float)width + eps);
  for (int c = threadIdx.x * V; c < width; c += EDGE_THREADS * V) {
    float v[V];
    EdgeVec<float, V>::load(xr + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= r;
    EdgeVec<T, V>::store(y + n * width + c, v);
  }
}

__global__ void sequence_advance_kernel(const long long* __restrict__ idx, int* __restrict__ pos, int* __restrict__ prev_token,
                                        const int* __restrict__ slots, const int* __restrict__ count, int B, int T) {
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= B || count[b] <= 0) return;
  pos[slots[b]] += count[b];
  prev_token[slots[b]] = (int)idx[(long long)b * T + count[b] - 1];
}

// tokens one CTA walks over: enough CTAs to fill the device first, then few recomputed rows
static int edge_run(int B, int T) {
  const long long n = (long long)B * T;
  long long run = n / (148 * 8);
  return (int)(run < 1 ? 1 : (run > 16 ? 16 : run));
}

template <typename T, int V, bool EMBED>
static int edge_launch(EdgeParams& p, cudaStream_t s) {
  p.run = edge_run(p.B, p.T);
  const dim3 grid((p.T + p.run - 1) / p.run, p.B);
  const bool late_state = p.gain && p.shift && p.T > 1;
  const float* x = EMBED ? p.hist : p.x_out;
#define KVB_EDGE(TH, NC)                                                                                                   \
  do {                                                                                                                     \
    layer_edge_kernel<T, V, TH, NC, EMBED><<<grid, TH, 0, s>>>(p);                                                         \
    if (late_state)                                                                                                        \
      shift_state_kernel<V, TH, NC><<<p.B, TH, 0, s>>>(x, p.gain, p.state, p.slots, p.count, p.T, p.width, p.eps);         \
  } while (0)
  if (p.width <= 256 * V) KVB_EDGE(256, 1);
  else if (p.width <= 512 * V) KVB_EDGE(512, 1);
  else if (p.width <= 1024 * V) KVB_EDGE(256, 4);
  else if (p.width <= 2048 * V) KVB_EDGE(512, 4);
  else return KVB_ERR_TOO_LARGE;
#undef KVB_EDGE
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <bool EMBED>
static int edge_dispatch(EdgeParams& p, int dtype, cudaStream_t s) {
  if (p.B <= 0 || p.T <= 0 || p.width <= 0 || p.B > 65535) return KVB_ERR_ARG;
  const bool vec = p.width % 4 == 0 && (p.expert_out == nullptr || p.expert_ld % 4 == 0);
  if (dtype == 0) return vec ? edge_launch<float, 4, EMBED>(p, s) : edge_launch<float, 1, EMBED>(p, s);
  if (dtype == 1) return vec ? edge_launch<__nv_bfloat16, 4, EMBED>(p, s) : edge_launch<__nv_bfloat16, 1, EMBED>(p, s);
  return KVB_ERR_ARG;
}

}  // namespace kvb

extern "C" int kvb_embed_edge(const long long* idx, const int* prev_token, const void* embed, const void* bigram, long long buckets,
                              long long mul_prev, long long mul_cur, float* hist, const float* gain, const float* shift, float* state,
                              void* h, void* hs, const int* slots, const int* start, const int* count, int B, int T, int width,
                              long long vocab, float eps, int dtype, int* status, void* stream) {
  kvb::EdgeParams p = {};
  p.vocab = vocab; p.status = status;
  p.idx = idx; p.prev_token = prev_token; p.embed = embed; p.bigram = bigram;
  p.buckets = buckets; p.mul_prev = mul_prev; p.mul_cur = mul_cur;
  p.hist = hist; p.gain = gain; p.shift = shift; p.state = state; p.h = h; p.hs = hs;
  p.slots = slots; p.start = start; p.count = count; p.B = B; p.T = T; p.width = width; p.eps = eps;
  if (bigram && buckets <= 0) return KVB_ERR_ARG;
  return kvb::edge_dispatch<true>(p, dtype, (cudaStream_t)stream);
}

extern "C" int kvb_layer_edge(const float* x_in, const void* mix, const void* expert_out, const int* expert_row, const float* expert_w,
                              int top, long long expert_ld, float* hist, int n_hist, long long hist_stride, const float* coef,
                              float* x_out, const float* gain, const float* shift, float* state, void* h, void* hs, const int* slots,
                              const int* start, const int* count, int B, int T, int width, float eps, int dtype, void* stream) {
  kvb::EdgeParams p = {};
  p.x_in = x_in; p.mix = mix; p.expert_out = expert_out; p.expert_row = expert_row; p.expert_w = expert_w; p.top = top;
  p.expert_ld = expert_ld; p.hist = hist; p.n_hist = n_hist; p.hist_stride = hist_stride; p.coef = coef; p.x_out = x_out;
  p.gain = gain; p.shift = shift; p.state = state; p.h = h; p.hs = hs;
  p.slots = slots; p.start = start; p.count = count; p.B = B; p.T = T; p.width = width; p.eps = eps;
  if (x_out == x_in) return KVB_ERR_ARG;
  return kvb::edge_dispatch<false>(p, dtype, (cudaStream_t)stream);
}

extern "C" int kvb_scalar_rmsnorm(const float* x, const long long* rows, const float* gain, void* y, long long n, int width, float eps,
                                  int dtype, void* stream) {
  if (n <= 0 || width <= 0 || n > 0x7fffffffLL) return KVB_ERR_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  const unsigned g = (unsigned)n;
  const bool vec = width % 4 == 0;
  if (dtype == 0) {
    if (vec) kvb::scalar_rmsnorm_kernel<float, 4><<<g, kvb::EDGE_THREADS, 0, s>>>(x, rows, gain, (float*)y, width, eps);
    else kvb::scalar_rmsnorm_kernel<float, 1><<<g, kvb::EDGE_THREADS, 0, s>>>(x, rows, gain, (float*)y, width, eps);
  } else if (dtype == 1) {
    if (vec) kvb::scalar_rmsnorm_kernel<__nv_bfloat16, 4><<<g, kvb::EDGE_THREADS, 0, s>>>(x, rows, gain, (__nv_bfloat16*)y, width, eps);
    else kvb::scalar_rmsnorm_kernel<__nv_bfloat16, 1><<<g, kvb::EDGE_THREADS, 0, s>>>(x, rows, gain, (__nv_bfloat16*)y, width, eps);
  } else {
    return KVB_ERR_ARG;
  }
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_sequence_advance(const long long* idx, int* pos, int* prev_token, const int* slots, const int* count, int B, int T,
                                    void* stream) {
  if (B <= 0 || T <= 0) return KVB_ERR_ARG;
  kvb::sequence_advance_kernel<<<(B + 127) / 128, 128, 0, (cudaStream_t)stream>>>(idx, pos, prev_token, slots, count, B, T);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
