// What happens between two sublayers of a model whose layers have norms before and / or after each sublayer, in one pass over
// the fp32 residual stream: weighted sum of a token's routed experts, norm of the sublayer's output, residual sum, what a loop adds
// ahead of a pass (embedding row of the token, a vector), norm for the next sublayer (or the stream itself, where sublayers read
// that). Also the entry into the stack (embedding rows only) and the norm of rows in front of the output head.
//
// A CTA has one row, which stays in registers; means and squared deviations are separate sums (no cancellation).
//
// What a sublayer reads may pass a short causal convolution over time first. A single token finds the inputs before it in a ring of its
// sequence. Of several tokens a CTA takes a run, one after the other, and keeps the inputs of the last ones in registers; those of the tokens
// right before the run are worked out once more. (Convolutions of more than eight taps and wide rows keep them in shared memory, some rows at a
// time, one per team of warps.)
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
  int run;  // tokens of a CTA
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

// columns [c, c + V) of h of a single token become h + its convolution; the ring takes h (its row is none of those that are read)
template <int V>
__device__ __forceinline__ void conv_single(const NormEdgeParams& p, int b, int c, float (&h)[V]) {
  const int taps = p.tok.taps, pos = p.tok.start[b];
  float* ring = p.tok.conv_ring + (long long)p.tok.slots[b] * taps * p.width + c;
  float w[V], v[V], s[V];
  RowVec<float, V>::load(p.tok.conv_w + (long long)(taps - 1) * p.width + c, w);
#pragma unroll
  for (int e = 0; e < V; ++e) s[e] = fmaf(w[e], h[e], h[e]);
#pragma unroll 4
  for (int k = 1; k < taps; ++k) {
    if (k > pos) break;
    RowVec<float, V>::load(p.tok.conv_w + (long long)(taps - 1 - k) * p.width + c, w);
    RowVec<float, V>::load(ring + (long long)((pos - k) % taps) * p.width, v);
#pragma unroll
    for (int e = 0; e < V; ++e) s[e] = fmaf(w[e], v[e], s[e]);
  }
  if (p.tok.count[b] > 0) RowVec<float, V>::store(ring + (long long)(pos % taps) * p.width, h);
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
  // columns of h, the convolution of a single token included; then out
  auto put_h = [&](int c, float (&w)[V]) {
    if (p.tok.conv_w && p.tok.T == 1) conv_single<V>(p, (int)n, c, w);
    RowVec<T, V>::store(static_cast<T*>(p.h) + o + c, w);
  };
  if (!p.before) {
    if (!p.h) return;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = (i * TH + threadIdx.x) * V;
      if (c < p.width) put_h(c, x[i]);
    }
    return;
  }
  r = row_norm_factor<TH, NC, V, CENTER>(x, p, red + 2);
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = (i * TH + threadIdx.x) * V;
    if (c >= p.width) continue;
    float w[V];
    RowVec<float, V>::load(p.before + c, w);
#pragma unroll
    for (int e = 0; e < V; ++e) w[e] *= x[i][e] * r;
    put_h(c, w);
  }
}

// ------------------------------------------------------------------------- several tokens with a convolution
// TAPS: taps that are kept in registers; a shorter convolution has zeros in front
template <typename T, int V, int TH, int NC, int TAPS, bool CENTER>
__global__ void __launch_bounds__(TH, TH == 128 ? 6 : TH == 256 ? 3 : 1)
conv_run_kernel(const NormEdgeParams p) {
  __shared__ float red[2][4][TH / 32];  // sums of a token, two tokens in turn
  const int T_ = p.tok.T, taps = p.tok.taps, b = blockIdx.y, t0 = blockIdx.x * p.run, t1 = min(t0 + p.run, T_);
  const int start = p.tok.start[b], count = p.tok.count[b], col = threadIdx.x * V;
  constexpr int STRIDE = TH * V;
  float* const ring = p.tok.conv_ring + (long long)p.tok.slots[b] * taps * p.width + col;
  const long long row0 = (long long)b * T_;
  float x[NC][V], y[NC][V], past[TAPS > 1 ? TAPS - 1 : 1][NC][V];  // past[k]: h of the token TAPS - 1 - k before
  auto fetch = [&](int t) {  // what row t of the pass is made of, on its way
    const long long o = (row0 + t) * p.width + col;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = y[i][e] = 0.f;
      if (col + i * STRIDE >= p.width) continue;
      if (p.sub) RowVec<T, V>::load(static_cast<const T*>(p.sub) + o + i * STRIDE, y[i]);
      if (p.x_in) RowVec<float, V>::load(p.x_in + o + i * STRIDE, x[i]);
    }
  };
  // the row of the stream (stored if `out`) in x, then its h
  auto work = [&](int t, bool out, float (&h)[NC][V], int next) {
    float (*r2)[TH / 32] = red[t & 1];
    const long long n = row0 + t, o = n * p.width + col;
    long long tok = 0;
    if (p.embed) {
      tok = p.idx[n];
      if (tok < 0 || tok >= p.vocab) {
        if (p.status) atomicCAS(p.status, 0, STATUS_BAD_INDEX);
        tok = 0;
      }
    }
    const float r = p.after ? row_norm_factor<TH, NC, V, CENTER>(y, p, r2) : 1.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = col + i * STRIDE;
      if (c >= p.width) {
#pragma unroll
        for (int e = 0; e < V; ++e) h[i][e] = 0.f;
        continue;
      }
      float w[V];
      if (p.after) {
        RowVec<float, V>::load(p.after + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) h[i][e] = fmaf(y[i][e] * r, w[e], x[i][e]);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) h[i][e] = x[i][e] + y[i][e];
      }
      if (p.embed) {
        RowVec<T, V>::load(static_cast<const T*>(p.embed) + tok * p.width + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) h[i][e] += w[e];
      }
      if (p.tok.table) {
        RowVec<T, V>::load(static_cast<const T*>(p.tok.table) + table_row(p, n) * p.width + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) h[i][e] += w[e];
      }
      if (p.step) {
        RowVec<float, V>::load(p.step + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) h[i][e] += w[e];
      }
      if (out && p.x_out) RowVec<float, V>::store(p.x_out + o + i * STRIDE, h[i]);
    }
    if (next >= 0) fetch(next);
    if (!p.before) return;
    const float f = row_norm_factor<TH, NC, V, CENTER>(h, p, r2 + 2);
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      if (col + i * STRIDE >= p.width) continue;
      float w[V];
      RowVec<float, V>::load(p.before + col + i * STRIDE, w);
#pragma unroll
      for (int e = 0; e < V; ++e) h[i][e] *= f * w[e];
    }
  };
  const int first = t0 - taps + 1;
  float h[NC][V];
  fetch(max(first, 0));
  for (int t = first; t < t1; ++t) {
    if (t >= 0) {
      work(t, t >= t0, h, t + 1 < t1 ? t + 1 : -1);
    } else {  // before the pass, perhaps before the sequence
#pragma unroll
      for (int i = 0; i < NC; ++i) {
#pragma unroll
        for (int e = 0; e < V; ++e) h[i][e] = 0.f;
        if (start + t >= 0 && col + i * STRIDE < p.width) RowVec<float, V>::load(ring + (long long)((start + t) % taps) * p.width + i * STRIDE, h[i]);
      }
    }
    if (t >= t0) {
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int c = col + i * STRIDE;
        if (c >= p.width) continue;
        float s[V], w[V];
        RowVec<float, V>::load(p.tok.conv_w + (long long)(taps - 1) * p.width + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] = fmaf(w[e], h[i][e], h[i][e]);
#pragma unroll
        for (int k = TAPS - 2; k >= 0; --k) {
          const int at = k - (TAPS - taps);
          if (at < 0) break;
          RowVec<float, V>::load(p.tok.conv_w + (long long)at * p.width + c, w);
#pragma unroll
          for (int e = 0; e < V; ++e) s[e] = fmaf(w[e], past[k][i][e], s[e]);
        }
        RowVec<T, V>::store(static_cast<T*>(p.h) + (row0 + t) * p.width + c, s);
      }
    }
#pragma unroll
    for (int i = 0; i < NC; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) {
#pragma unroll
        for (int k = 0; k + 2 < TAPS; ++k) past[k][i][e] = past[k + 1][i][e];
        if (TAPS > 1) past[TAPS - 2][i][e] = h[i][e];
      }
  }
  // the ring takes the last ones of the sequence. Only the CTA of the first tokens has read it, so it alone may write there
  if (t0 > 0) return;
  for (int t = max(0, count - taps); t < count; ++t) {
    fetch(t);
    __syncthreads();  // sums of the tokens before have been read
    work(t, false, h, -1);
#pragma unroll
    for (int i = 0; i < NC; ++i)
      if (col + i * STRIDE < p.width) RowVec<float, V>::store(ring + (long long)((start + t) % taps) * p.width + i * STRIDE, h[i]);
  }
}

template <typename T, int V, int TH, int NC, bool CENTER>
static int conv_run_launch(NormEdgeParams& p, int B, cudaStream_t s) {
  // a wave of CTAs, but no runs so short that most of the work is done twice
  const int per_sm = TH == 128 ? 6 : TH == 256 ? 3 : 1;
  long long runs = (148LL * per_sm) / B;
  const long long most = (p.tok.T + 15) / 16;
  if (runs > most) runs = most;
  if (runs < 1) runs = 1;
  p.run = (int)((p.tok.T + runs - 1) / runs);
  if (p.run > 64) p.run = 64;  // many waves: even ends
  if (p.run < p.tok.taps) p.run = p.tok.taps;
  const dim3 grid((p.tok.T + p.run - 1) / p.run, B);
  if (p.tok.taps <= 4) conv_run_kernel<T, V, TH, NC, 4, CENTER><<<grid, TH, 0, s>>>(p);
  else conv_run_kernel<T, V, TH, NC, 8, CENTER><<<grid, TH, 0, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <typename T, bool CENTER>
static int conv_run_type(NormEdgeParams& p, int B, cudaStream_t s) {
  if (p.width % 4) {
    if (p.width <= 1024) return conv_run_launch<T, 1, 256, 4, CENTER>(p, B, s);
    return KVB_ERR_TOO_LARGE;
  }
  if (p.width <= 512) return conv_run_launch<T, 4, 128, 1, CENTER>(p, B, s);
  if (p.width <= 1024) return conv_run_launch<T, 4, 256, 1, CENTER>(p, B, s);
  if (p.width <= 2048) return conv_run_launch<T, 4, 256, 2, CENTER>(p, B, s);
  if (p.width <= 4096) return conv_run_launch<T, 4, 512, 2, CENTER>(p, B, s);
  return KVB_ERR_TOO_LARGE;
}

constexpr int CE_WARPS = 8;

// sums over the lanes of a team of `tw` warps (every warp of the CTA calls)
__device__ __forceinline__ float team_sum(float v, int tw, float* red) {
  v = warp_sum(v);
  if (tw == 1) return v;
  const int warp = threadIdx.x >> 5;
  if ((threadIdx.x & 31) == 0) red[warp] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < tw; ++i) s += red[warp / tw * tw + i];
  return s;
}

// NC accesses of V columns per lane; a row has tw warps (a power of two), so CE_WARPS / tw rows are worked on side by side. Shared memory: h of
// these rows and of the taps - 1 before them, the row of token t in place (t + taps - 1) mod their number.
template <typename T, int V, int NC, bool CENTER>
__global__ void __launch_bounds__(CE_WARPS * 32)
conv_edge_kernel(const NormEdgeParams p, int tw) {
  extern __shared__ float ce_h[];
  __shared__ float red[4][CE_WARPS];
  const int T_ = p.tok.T, taps = p.tok.taps, rows = CE_WARPS / tw, places = rows + taps - 1;
  const int b = blockIdx.y, t0 = blockIdx.x * p.run, t1 = min(t0 + p.run, T_);
  const int start = p.tok.start[b], count = p.tok.count[b];
  const int team = (threadIdx.x >> 5) / tw, col = (threadIdx.x - team * tw * 32) * V, stride = tw * 32 * V;
  float* ring = p.tok.conv_ring + (long long)p.tok.slots[b] * taps * p.width;
  float x[NC][V], y[NC][V];
  // what row t of the pass is made of, on its way
  auto fetch = [&](int t) {
    const long long o = ((long long)b * T_ + t) * p.width;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = col + i * stride;
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = y[i][e] = 0.f;
      if (c >= p.width || t < 0 || t >= T_) continue;
      if (p.sub) RowVec<T, V>::load(static_cast<const T*>(p.sub) + o + c, y[i]);
      if (p.x_in) RowVec<float, V>::load(p.x_in + o + c, x[i]);
    }
  };
  auto factor = [&](float (&v)[NC][V], float (*r)[CE_WARPS]) {
    if (CENTER) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < NC; ++i)
#pragma unroll
        for (int e = 0; e < V; ++e) s += v[i][e];
      const float mean = team_sum(s, tw, r[0]) * p.inv_width;
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (col + i * stride < p.width) {
#pragma unroll
          for (int e = 0; e < V; ++e) v[i][e] -= mean;
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[i][e], v[i][e], ss);
    return 1.f / sqrtf(team_sum(ss, tw, r[1]) * p.inv_width + p.eps);
  };
  // from what fetch brought to the row of the stream (stored if `out`) and its h in registers; all threads take part
  auto work = [&](int t, bool out) {
    const long long n = (long long)b * T_ + t, o = n * p.width;
    const bool in = t >= 0 && t < T_;
    long long tok = 0;
    if (p.embed && in) {
      tok = p.idx[n];
      if (tok < 0 || tok >= p.vocab) {
        if (p.status) atomicCAS(p.status, 0, STATUS_BAD_INDEX);
        tok = 0;
      }
    }
    const float r = p.after ? factor(y, red) : 1.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = col + i * stride;
      if (c >= p.width || !in) continue;
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
      if (out && p.x_out) RowVec<float, V>::store(p.x_out + o + c, x[i]);
    }
    if (!p.before) return;
    const float f = factor(x, red + 2);
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = col + i * stride;
      if (c >= p.width) continue;
      float w[V];
      RowVec<float, V>::load(p.before + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] *= f * w[e];
    }
  };
  auto place = [&](int t) { return ce_h + (t + taps - 1) % places * p.width; };
  for (int base = t0 - taps + 1; base < t1; base += rows) {
    const int t = base + team;
    const bool mine = t < t1, past = t < 0;
    if (base == t0 - taps + 1) fetch(mine ? t : -1);
    work(mine ? t : -1, t >= t0);
    if (mine) {
      const bool held = past && start + t >= 0;
      float* d = place(t);
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int c = col + i * stride;
        if (c >= p.width) continue;
        if (past) {
#pragma unroll
          for (int e = 0; e < V; ++e) x[i][e] = 0.f;
          if (held) RowVec<float, V>::load(ring + (long long)((start + t) % taps) * p.width + c, x[i]);
        }
        RowVec<float, V>::store(d + c, x[i]);
      }
    }
    fetch(t + rows < t1 ? t + rows : -1);
    __syncthreads();
    // every thread has its columns of up to four rows: weights are read once for them
    const int end = min(base + rows, t1);
    for (int u0 = max(base, t0); u0 < end; u0 += 4) {
      for (int c = threadIdx.x * V; c < p.width; c += CE_WARPS * 32 * V) {
        float s[4][V], w[V], h[V];
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (u0 + j < end) RowVec<float, V>::load(place(u0 + j) + c, s[j]);
        for (int k = 0; k < taps; ++k) {
          RowVec<float, V>::load(p.tok.conv_w + (long long)k * p.width + c, w);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            if (u0 + j >= end) break;
            RowVec<float, V>::load(place(u0 + j - taps + 1 + k) + c, h);
#pragma unroll
            for (int e = 0; e < V; ++e) s[j][e] = fmaf(w[e], h[e], s[j][e]);
          }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (u0 + j < end) RowVec<T, V>::store(static_cast<T*>(p.h) + ((long long)b * T_ + u0 + j) * p.width + c, s[j]);
      }
    }
    __syncthreads();
  }
  // the ring takes the last ones of the sequence. Only the CTA of the first tokens has read it, so it alone may write there
  if (t0 > 0 || count <= 0) return;
  for (int base = max(0, count - taps); base < count; base += rows) {
    const int t = base + team;
    fetch(t < count ? t : -1);
    __syncthreads();  // the sums of the rows before have been read
    work(t < count ? t : -1, false);
    if (t >= count) continue;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = col + i * stride;
      if (c < p.width) RowVec<float, V>::store(ring + (long long)((start + t) % taps) * p.width + c, x[i]);
    }
  }
}

template <typename T, int V, int NC, bool CENTER>
static int conv_edge_launch(NormEdgeParams& p, long long n, cudaStream_t s) {
  int tw = 1;
  while (tw < CE_WARPS && tw * 32 * V * NC < p.width) tw *= 2;
  if (tw * 32 * V * NC < p.width) return KVB_ERR_TOO_LARGE;
  const int rows = CE_WARPS / tw, B = (int)(n / p.tok.T);
  const size_t smem = (size_t)(rows + p.tok.taps - 1) * p.width * sizeof(float);
  if (smem > 220 * 1024) return KVB_ERR_TOO_LARGE;
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(conv_edge_kernel<T, V, NC, CENTER>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  // a wave of CTAs, but no runs so short that most of the work is done twice
  const int per_sm = smem > 110 * 1024 ? 1 : smem > 72 * 1024 ? 2 : 3;
  long long runs = (148LL * per_sm + B - 1) / B;
  const long long most = (p.tok.T + 4 * (p.tok.taps - 1) + rows - 1) / (4 * (p.tok.taps - 1) + rows);
  if (runs > most) runs = most;
  p.run = (int)((p.tok.T + runs - 1) / runs);
  conv_edge_kernel<T, V, NC, CENTER><<<dim3((p.tok.T + p.run - 1) / p.run, B), CE_WARPS * 32, smem, s>>>(p, tw);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <typename T>
static int conv_edge_type(NormEdgeParams& p, long long n, int center, cudaStream_t s) {
  if (p.width % 4) return center ? conv_edge_launch<T, 1, 32, true>(p, n, s) : conv_edge_launch<T, 1, 32, false>(p, n, s);
  return center ? conv_edge_launch<T, 4, 8, true>(p, n, s) : conv_edge_launch<T, 4, 8, false>(p, n, s);
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
                 (tokens->conv_w && (!tokens->conv_ring || tokens->taps <= 0 || !h || (tokens->T > 1 && (x_out == x_in || expert_out))))))
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
  p.run = 0;
  if (tokens && tokens->conv_w && tokens->T > 1) {
    if (tokens->taps <= 8 && width <= (width % 4 ? 1024 : 4096)) {
      const int B = (int)(n / tokens->T);
      cudaStream_t s = (cudaStream_t)stream;
      if (dtype == 0) return center ? kvb::conv_run_type<float, true>(p, B, s) : kvb::conv_run_type<float, false>(p, B, s);
      if (dtype == 1) return center ? kvb::conv_run_type<__nv_bfloat16, true>(p, B, s) : kvb::conv_run_type<__nv_bfloat16, false>(p, B, s);
      return KVB_ERR_ARG;
    }
    if (dtype == 0) return kvb::conv_edge_type<float>(p, n, center, (cudaStream_t)stream);
    if (dtype == 1) return kvb::conv_edge_type<__nv_bfloat16>(p, n, center, (cudaStream_t)stream);
    return KVB_ERR_ARG;
  }
  if (dtype == 0) return kvb::norm_edge_type<float>(p, n, center, (cudaStream_t)stream);
  if (dtype == 1) return kvb::norm_edge_type<__nv_bfloat16>(p, n, center, (cudaStream_t)stream);
  return KVB_ERR_ARG;
}
