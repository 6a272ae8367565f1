// State-space (Mamba-2) mixers: short causal convolution, recurrence, gated norm in parts; and the activation of dense
// feed-forwards.
//
//   conv   x, B and C of several new tokens: convolution per channel with bias and silu. The inputs before the pass lie in a
//          ring of `taps` rows per sequence (position p in row p mod taps);
//   scan   the recurrence token by token on CUDA cores (fp32, and shapes that the chunked kernel of ssm_sm100.cu does not take);
//   step   one new token per sequence: convolution, step size, decay, state and output of a head in one kernel, bound by
//          reading and writing the state once;
//   norm   y · silu(z), divided by the root mean square of each part.
//
// States are fp32, (slots, heads, np, vdp). A sequence that starts at position 0 reads neither state nor ring. Rows without
// tokens and padding change nothing; their outputs are zero or finite.
#include "common.cuh"
#include "kvb200_layers.h"
#include "ssm.cuh"

namespace kvb {

template <typename T, int V>
struct alignas(sizeof(T) * V) SsVec {
  T v[V];
};

// ------------------------------------------------------------------------------------------------ conv
constexpr int SC_THREADS = 128;
constexpr int SC_RUN = 32;  // tokens of a thread

struct ConvParams {
  const float *w, *bias;  // (taps, channels), (channels)
  const int *slots, *start, *count;
  long long ld;
  int T, col, channels, taps, run, silu;
};

// TAPS 0: any number, inputs are read once per tap
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(SC_THREADS)
short_conv_kernel(const T* __restrict__ u, T* __restrict__ out, T* __restrict__ ring, const ConvParams p) {
  using Vec = SsVec<T, V>;
  const int c = (blockIdx.x * SC_THREADS + threadIdx.x) * V, b = blockIdx.z;
  if (c >= p.channels) return;
  const int t0 = blockIdx.y * p.run, t1 = min(t0 + p.run, p.T);
  const int start = p.start[b], taps = TAPS ? TAPS : p.taps;
  const T* src = u + (long long)b * p.T * p.ld + p.col + c;
  T* dst = out + (long long)b * p.T * p.channels + c;
  T* past = ring + (long long)p.slots[b] * taps * p.channels + c;
  // input of token t of the pass, possibly before it
  auto input = [&](int t, float (&x)[V]) {
    Vec a;
    if (t >= 0) {
      a = *reinterpret_cast<const Vec*>(src + (long long)t * p.ld);
    } else if (start + t >= 0) {
      a = *reinterpret_cast<const Vec*>(past + (long long)((start + t) % taps) * p.channels);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) a.v[e] = from_f32<T>(0.f);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = to_f32(a.v[e]);
  };
  float bias[V];
#pragma unroll
  for (int e = 0; e < V; ++e) bias[e] = p.bias ? p.bias[c + e] : 0.f;
  if constexpr (TAPS > 0) {
    float w[TAPS][V], x[TAPS][V];
#pragma unroll
    for (int k = 0; k < TAPS; ++k)
#pragma unroll
      for (int e = 0; e < V; ++e) w[k][e] = p.w[(long long)k * p.channels + c + e];
#pragma unroll
    for (int k = 0; k < TAPS - 1; ++k) input(t0 - TAPS + 1 + k, x[k + 1]);
    constexpr int AHEAD = 8;
    for (int t = t0; t < t1; t += AHEAD) {
      Vec next[AHEAD];
#pragma unroll
      for (int i = 0; i < AHEAD; ++i)
        if (t + i < t1) next[i] = *reinterpret_cast<const Vec*>(src + (long long)(t + i) * p.ld);
#pragma unroll
      for (int i = 0; i < AHEAD; ++i) {
        if (t + i >= t1) break;
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
          for (int e = 0; e < V; ++e) x[k][e] = x[k + 1][e];
        Vec y;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          x[TAPS - 1][e] = to_f32(next[i].v[e]);
          float acc = bias[e];
#pragma unroll
          for (int k = 0; k < TAPS; ++k) acc = fmaf(w[k][e], x[k][e], acc);
          y.v[e] = from_f32<T>(p.silu ? ss_silu_for<T>(acc) : acc);
        }
        *reinterpret_cast<Vec*>(dst + (long long)(t + i) * p.channels) = y;
      }
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float acc[V], x[V];
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = bias[e];
      for (int k = 0; k < taps; ++k) {
        input(t - taps + 1 + k, x);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(p.w[(long long)k * p.channels + c + e], x[e], acc[e]);
      }
      Vec y;
#pragma unroll
      for (int e = 0; e < V; ++e) y.v[e] = from_f32<T>(p.silu ? ss_silu_for<T>(acc[e]) : acc[e]);
      *reinterpret_cast<Vec*>(dst + (long long)t * p.channels) = y;
    }
  }
  // only the thread of the first tokens reads the ring of its channels, so it alone may write there
  if (t0 == 0) {
    const int n = p.count[b];
    for (int t = max(0, n - taps); t < n; ++t)
      *reinterpret_cast<Vec*>(past + (long long)((start + t) % taps) * p.channels) = *reinterpret_cast<const Vec*>(src + (long long)t * p.ld);
  }
}

template <typename T, int V>
static int conv_launch_vec(const void* u, void* out, void* ring, ConvParams& p, int B, cudaStream_t s) {
  const int blocks = (p.channels / V + SC_THREADS - 1) / SC_THREADS;
  long long run = ((long long)p.T * B * blocks + 148 * 8 - 1) / (148 * 8);  // a wave of CTAs first, then few inputs read twice
  p.run = (int)(run < 4 ? 4 : (run > SC_RUN ? SC_RUN : (run + 7) / 8 * 8));
  if (p.run < p.taps) p.run = p.taps;  // only the first run of a channel may look back beyond the pass
  const dim3 grid(blocks, (p.T + p.run - 1) / p.run, B);
  if (p.taps == 4) short_conv_kernel<T, V, 4><<<grid, SC_THREADS, 0, s>>>((const T*)u, (T*)out, (T*)ring, p);
  else short_conv_kernel<T, V, 0><<<grid, SC_THREADS, 0, s>>>((const T*)u, (T*)out, (T*)ring, p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <typename T>
static int conv_launch(const void* u, void* out, void* ring, ConvParams& p, int B, cudaStream_t s) {
  if (p.channels % 4 || p.col % 4 || p.ld % 4) return conv_launch_vec<T, 1>(u, out, ring, p, B, s);
  return conv_launch_vec<T, 4>(u, out, ring, p, B, s);
}

// ------------------------------------------------------------------------------------------------ scan
constexpr int SN_COLS = 32;   // value columns of a CTA
constexpr int SN_ROWS = 8;    // rows of the state that are worked on side by side
constexpr int SN_CHUNK = 8;   // tokens staged at a time

// Decays of their own for every row of the state (gated linear attention), from the same input as B and C.
struct RowDecay {
  kvb_gated_linear g;
  const int* only;  // heads of rows of the pass to work on, NULL: all
};

// NR: rows of the state per thread; thread (p, r) has column p of rows r, r + SN_ROWS, ... TB: type of B and C; BY_ROW: decays by row, and C is
// scaled
template <typename T, typename TB, int NR, bool BY_ROW>
__global__ void __launch_bounds__(SN_COLS * SN_ROWS)
state_scan_simple_kernel(const T* __restrict__ u, const T* __restrict__ x, long long ldx, const TB* __restrict__ bm, const TB* __restrict__ cm,
                         long long ldb, T* __restrict__ y, const ScanParams p, const RowDecay rd) {
  constexpr int NP = NR * SN_ROWS;
  constexpr int SN_CHUNK = BY_ROW ? 4 : kvb::SN_CHUNK;
  __shared__ float srow[BY_ROW ? SN_CHUNK : 1][BY_ROW ? NP : 1];
  if (BY_ROW && rd.only && !rd.only[blockIdx.z * p.heads + blockIdx.y]) return;
  __shared__ float sb[SN_CHUNK][NP], sc[SN_CHUNK][NP], sx[SN_CHUNK][SN_COLS], sdt[SN_CHUNK], sa[SN_CHUNK];
  __shared__ float part[SN_CHUNK][SN_ROWS][SN_COLS];
  const int p0 = blockIdx.x * SN_COLS, h = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, col = tid % SN_COLS, r = tid / SN_COLS;
  const int g = h / (p.heads / p.groups), n = p.count[b];
  const bool mine = p0 + col < p.vdp;
  float* st = p.state + ((long long)p.slots[b] * p.heads + h) * p.np * p.vdp + p0 + col;
  float s[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = r + i * SN_ROWS;
    s[i] = p.start[b] > 0 && mine && row < p.np ? st[(long long)row * p.vdp] : 0.f;
  }
  const bool fixed = BY_ROW || p.decay;
  const float rate = fixed ? 0.f : -expf(p.a_log[h]), skip = fixed ? 0.f : p.skip[h], bias = fixed ? 0.f : p.dt_bias[h];
  x += (long long)b * p.T * ldx;
  bm += (long long)b * p.T * ldb;
  cm += (long long)b * p.T * ldb;
  for (int t0 = 0; t0 < p.T; t0 += SN_CHUNK) {
    const int nt = min(SN_CHUNK, p.T - t0);
    for (int i = tid; i < nt * NP; i += SN_COLS * SN_ROWS) {
      const int t = i / NP, k = i - t * NP;
      const long long at = (long long)(t0 + t) * ldb + g * p.np + k;
      sb[t][k] = k < p.np ? to_f32(bm[at]) : 0.f;
      sc[t][k] = k < p.np ? to_f32(cm[at]) * (BY_ROW ? rd.g.q_scale : 1.f) : 0.f;
      if constexpr (BY_ROW) {
        float d = 0.f;
        if (k < p.np) d = ss_decay(gl_log_decay(rd.g, rd.g.in + ((long long)b * p.T + t0 + t) * rd.g.ld + 2 * rd.g.heads * p.np, h * p.np + k));
        srow[t][k] = d;
      }
    }
    for (int i = tid; i < nt * SN_COLS; i += SN_COLS * SN_ROWS) {
      const int t = i / SN_COLS, k = i - t * SN_COLS;
      sx[t][k] = p0 + k < p.vdp ? to_f32(x[(long long)(t0 + t) * ldx + h * p.vdp + p0 + k]) : 0.f;
    }
    if (tid < nt && fixed) {
      sdt[tid] = 1.f;
      sa[tid] = BY_ROW ? 0.f : p.decay[h];
    } else if (tid < nt) {
      const float dt = ss_softplus(to_f32(u[((long long)b * p.T + t0 + tid) * p.ld + p.dt_col + h]) + bias);
      sdt[tid] = dt;
      sa[tid] = ss_decay(rate * dt);
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      float acc = 0.f;
      if (t0 + t < n) {
        const float a = sa[t], dx = sdt[t] * sx[t][col];
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          s[i] = fmaf(BY_ROW ? srow[t][r + i * SN_ROWS] : a, s[i], dx * sb[t][r + i * SN_ROWS]);
          acc = fmaf(s[i], sc[t][r + i * SN_ROWS], acc);
        }
      }
      part[t][r][col] = acc;
    }
    __syncthreads();
    for (int i = tid; i < nt * SN_COLS; i += SN_COLS * SN_ROWS) {
      const int t = i / SN_COLS, k = i - t * SN_COLS;
      if (p0 + k >= p.vdp) continue;
      float acc = t0 + t < n ? skip * sx[t][k] : 0.f;
#pragma unroll
      for (int j = 0; j < SN_ROWS; ++j) acc += part[t][j][k];
      y[((long long)b * p.T + t0 + t) * p.inner + h * p.vdp + p0 + k] = from_f32<T>(acc);
    }
    __syncthreads();
  }
  if (n <= 0 || !mine) return;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = r + i * SN_ROWS;
    if (row < p.np) st[(long long)row * p.vdp] = s[i];
  }
}

template <typename T, typename TB = T, bool BY_ROW = false>
static int scan_simple_launch(const void* u, const void* x, long long ldx, const void* bm, const void* cm, long long ldb, void* y,
                              const ScanParams& p, int B, cudaStream_t s, const RowDecay& rd = RowDecay{}) {
  const dim3 grid((p.vdp + SN_COLS - 1) / SN_COLS, p.heads, B);
#define KVB_SCAN(NR) state_scan_simple_kernel<T, TB, NR, BY_ROW><<<grid, SN_COLS * SN_ROWS, 0, s>>>( \
    (const T*)u, (const T*)x, ldx, (const TB*)bm, (const TB*)cm, ldb, (T*)y, p, rd)
  if (p.np <= 4 * SN_ROWS) KVB_SCAN(4);
  else if (p.np <= 16 * SN_ROWS) KVB_SCAN(16);
  else if (p.np <= 32 * SN_ROWS) KVB_SCAN(32);
  else if (p.np <= 64 * SN_ROWS) KVB_SCAN(64);
  else return KVB_ERR_TOO_LARGE;
#undef KVB_SCAN
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

// ------------------------------------------------------------------------------------------------ step
constexpr int SS_THREADS = 256;
constexpr int SS_BATCH = 8;  // float4 of the state that a thread has in flight

struct StepParams {
  ScanParams s;
  const float *w, *bias;
  int taps, col;
};

// One head of one sequence. Thread (row, quad) has four value columns of rows row, row + n_rows, ...
template <typename T>
__global__ void __launch_bounds__(SS_THREADS)
state_step_kernel(const T* __restrict__ u, T* __restrict__ ring, T* __restrict__ y, const StepParams q) {
  extern __shared__ float step_sm[];  // x (vdp) | B (np) | C (np) | partial sums (SS_THREADS · 4)
  const ScanParams& p = q.s;
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  T* yr = y + (long long)b * p.inner + h * p.vdp;
  if (p.count[b] <= 0) {
    for (int i = tid; i < p.vdp; i += SS_THREADS) yr[i] = from_f32<T>(0.f);
    return;
  }
  float *sx = step_sm, *sb = sx + p.vdp, *sc = sb + p.np, *part = sc + p.np;
  const int quads = p.vdp / 4, n_rows = SS_THREADS / quads;
  const int row0 = tid / quads, quad = tid - row0 * quads;
  const bool active = row0 < n_rows;
  const int start = p.start[b];
  float4* st = reinterpret_cast<float4*>(p.state + ((long long)p.slots[b] * p.heads + h) * p.np * p.vdp) + quad;
  float4 s[SS_BATCH];
  auto load = [&](int base) {
#pragma unroll
    for (int i = 0; i < SS_BATCH; ++i) {
      const int row = base + i * n_rows;
      s[i] = start > 0 && active && row < p.np ? __ldcs(st + (long long)row * quads) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(row0);  // on its way during the convolution
  const int g = h / (p.heads / p.groups);
  const bool writes_bc = h % (p.heads / p.groups) == 0;
  const T* ur = u + (long long)b * p.ld;
  T* past = ring + (long long)p.slots[b] * q.taps * p.channels;
  for (int i = tid; i < p.vdp + 2 * p.np; i += SS_THREADS) {
    int c;
    if (i < p.vdp) c = h * p.vdp + i;
    else if (i < p.vdp + p.np) c = p.inner + g * p.np + i - p.vdp;
    else c = p.inner + (p.groups + g) * p.np + i - p.vdp - p.np;
    const T now = ur[q.col + c];
    float acc = fmaf(q.w[(long long)(q.taps - 1) * p.channels + c], to_f32(now), q.bias[c]);
    for (int k = 1; k < q.taps; ++k)
      if (start - k >= 0)
        acc = fmaf(q.w[(long long)(q.taps - 1 - k) * p.channels + c], to_f32(past[(long long)((start - k) % q.taps) * p.channels + c]), acc);
    step_sm[i] = ss_silu(acc);
    // the ring has one row more than a step reads, so heads that share a group do not disturb each other
    if (i < p.vdp || writes_bc) past[(long long)(start % q.taps) * p.channels + c] = now;
  }
  const float dt = ss_softplus(to_f32(ur[p.dt_col + h]) + p.dt_bias[h]);
  const float a = ss_decay(-expf(p.a_log[h]) * dt);
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    const float4 xv = *reinterpret_cast<const float4*>(sx + 4 * quad);
    const float4 dx = make_float4(dt * xv.x, dt * xv.y, dt * xv.z, dt * xv.w);
    for (int base = row0;;) {
#pragma unroll
      for (int i = 0; i < SS_BATCH; ++i) {
        const int row = base + i * n_rows;
        if (row >= p.np) break;
        const float bn = sb[row], cn = sc[row];
        float4 v = s[i];
        v.x = fmaf(a, v.x, dx.x * bn);
        v.y = fmaf(a, v.y, dx.y * bn);
        v.z = fmaf(a, v.z, dx.z * bn);
        v.w = fmaf(a, v.w, dx.w * bn);
        __stcs(st + (long long)row * quads, v);
        acc.x = fmaf(v.x, cn, acc.x);
        acc.y = fmaf(v.y, cn, acc.y);
        acc.z = fmaf(v.z, cn, acc.z);
        acc.w = fmaf(v.w, cn, acc.w);
      }
      base += SS_BATCH * n_rows;
      if (base >= p.np) break;
      load(base);
    }
    *reinterpret_cast<float4*>(part + 4 * (row0 * quads + quad)) = acc;
  }
  __syncthreads();
  const float skip = p.skip[h];
  for (int i = tid; i < p.vdp; i += SS_THREADS) {
    float v = skip * sx[i];
    for (int r = 0; r < n_rows; ++r) v += part[r * p.vdp + i];
    yr[i] = from_f32<T>(v);
  }
}

// ------------------------------------------------------------------------------------------------ norm
constexpr int GN_THREADS = 128;

struct GroupNormParams {
  const float* weight;  // (inner), padded like y
  long long ld;         // of z
  int heads, vdim, vdp, size, inner;
  float eps;
};

// One part of one row. V > 1: heads have no padding, the part's columns are contiguous and stay in registers (NC accesses
// of V per thread); V 1: any sizes, read twice.
template <typename T, int V, int NC>
__global__ void __launch_bounds__(GN_THREADS)
gated_group_norm_kernel(const T* __restrict__ y, const T* __restrict__ z, T* __restrict__ out, const GroupNormParams p) {
  using Vec = SsVec<T, V>;
  __shared__ float red[GN_THREADS / 32];
  const int g = blockIdx.y;
  const long long n = blockIdx.x;
  y += n * p.inner;
  z += n * p.ld;
  out += n * p.inner;
  float v[NC][V];
  float ss = 0.f;
  auto column = [&](int i) {  // of coordinate i of the part
    const int c = g * p.size + i;
    return V > 1 ? c : c / p.vdim * p.vdp + c % p.vdim;
  };
  auto gated = [&](int c, float (&r)[V]) {
    const Vec a = *reinterpret_cast<const Vec*>(y + c), d = *reinterpret_cast<const Vec*>(z + c);
#pragma unroll
    for (int e = 0; e < V; ++e) r[e] = to_f32(a.v[e]) * ss_silu_for<T>(to_f32(d.v[e]));
  };
  if constexpr (V > 1) {
#pragma unroll
    for (int k = 0; k < NC; ++k) {
      const int i = (k * GN_THREADS + threadIdx.x) * V;
      if (i >= p.size) continue;
      gated(column(i), v[k]);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[k][e], v[k][e], ss);
    }
  } else {
    for (int i = threadIdx.x; i < p.size; i += GN_THREADS) {
      gated(column(i), v[0]);
      ss = fmaf(v[0][0], v[0][0], ss);
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < GN_THREADS / 32; ++i) ss += red[i];
  const float r = 1.f / sqrtf(ss / (float)p.size + p.eps);
  if constexpr (V > 1) {
#pragma unroll
    for (int k = 0; k < NC; ++k) {
      const int i = (k * GN_THREADS + threadIdx.x) * V;
      if (i >= p.size) continue;
      const int c = column(i);
      Vec o;
#pragma unroll
      for (int e = 0; e < V; ++e) o.v[e] = from_f32<T>(v[k][e] * r * p.weight[c + e]);
      *reinterpret_cast<Vec*>(out + c) = o;
    }
  } else {
    for (int i = threadIdx.x; i < p.size; i += GN_THREADS) {
      const int c = column(i);
      gated(c, v[0]);
      out[c] = from_f32<T>(v[0][0] * r * p.weight[c]);
    }
    if (g == 0) {  // padding of the heads
      const int pad = p.vdp - p.vdim;
      for (int i = threadIdx.x; i < p.heads * pad; i += GN_THREADS) out[i / pad * p.vdp + p.vdim + i % pad] = from_f32<T>(0.f);
    }
  }
}

template <typename T>
static int group_norm_launch(const void* y, const void* z, void* out, const GroupNormParams& p, int parts, long long n, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const dim3 grid((unsigned)n, parts);
#define KVB_GNORM(VV, NC) gated_group_norm_kernel<T, VV, NC><<<grid, GN_THREADS, 0, s>>>((const T*)y, (const T*)z, (T*)out, p)
  const int per = (p.size + GN_THREADS * V - 1) / (GN_THREADS * V);
  if (p.vdim == p.vdp && p.size % V == 0 && p.ld % V == 0 && per <= 8) {
    if (per <= 1) KVB_GNORM(V, 1);
    else if (per <= 2) KVB_GNORM(V, 2);
    else if (per <= 4) KVB_GNORM(V, 4);
    else KVB_GNORM(V, 8);
  } else {
    KVB_GNORM(1, 1);
  }
#undef KVB_GNORM
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

// ------------------------------------------------------------------------------------------ activation
template <typename T, int V>
__global__ void __launch_bounds__(256)
relu_squared_kernel(T* __restrict__ x, long long n) {
  const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * V;
  if (i + V <= n) {
    SsVec<T, V> a = *reinterpret_cast<const SsVec<T, V>*>(x + i);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float r = fmaxf(to_f32(a.v[e]), 0.f);
      a.v[e] = from_f32<T>(r * r);
    }
    *reinterpret_cast<SsVec<T, V>*>(x + i) = a;
  } else {
    for (long long k = i; k < n; ++k) {
      const float r = fmaxf(to_f32(x[k]), 0.f);
      x[k] = from_f32<T>(r * r);
    }
  }
}

}  // namespace kvb

#define KVB_SSM_TYPES(dtype, ...)                             \
  switch (dtype) {                                            \
    case 0: { using T = float; __VA_ARGS__; break; }          \
    case 1: { using T = __nv_bfloat16; __VA_ARGS__; break; }  \
    default: return KVB_ERR_ARG;                              \
  }

extern "C" int kvb_short_conv(const void* u, long long ld, int col, const float* w, const float* bias, void* out, void* ring,
                              const int* slots, const int* start, const int* count, int B, int T_, int channels, int taps, int silu,
                              int dtype, void* stream) {
  if (B <= 0 || B > 65535 || T_ <= 0 || channels <= 0 || taps <= 0) return KVB_ERR_ARG;
  kvb::ConvParams p;
  p.w = w; p.bias = bias; p.slots = slots; p.start = start; p.count = count; p.ld = ld; p.T = T_; p.col = col; p.channels = channels;
  p.taps = taps; p.silu = silu;
  KVB_SSM_TYPES(dtype, return kvb::conv_launch<T>(u, out, ring, p, B, (cudaStream_t)stream));
}

extern "C" int kvb_state_scan(const void* u, long long ld, int dt_col, const void* xbc, const float* dt_bias, const float* a_log,
                              const float* skip, float* state, void* y, const int* slots, const int* start, const int* count, int B,
                              int T_, int heads, int groups, int vdp, int np, int dtype, void* stream) {
  if (B <= 0 || B > 65535 || T_ <= 0 || heads <= 0 || heads > 65535 || groups <= 0 || heads % groups || vdp <= 0 || np <= 0) return KVB_ERR_ARG;
  kvb::ScanParams p;
  p.dt_bias = dt_bias; p.a_log = a_log; p.skip = skip; p.decay = nullptr; p.slots = slots; p.start = start; p.count = count;
  p.state = state; p.ld = ld; p.T = T_; p.dt_col = dt_col; p.heads = heads; p.groups = groups; p.vdp = vdp; p.np = np; p.inner = heads * vdp;
  p.channels = heads * vdp + 2 * groups * np;
  KVB_SSM_TYPES(dtype, const T* x = (const T*)xbc; const T* bm = x + p.inner;
                return kvb::scan_simple_launch<T>(u, x, p.channels, bm, bm + groups * np, p.channels, y, p, B, (cudaStream_t)stream));
}

extern "C" int kvb_retention_scan(const void* v, long long ldv, const void* qk, long long ldqk, const float* decay, float* state, void* y,
                                  const int* slots, const int* start, const int* count, int B, int T_, int heads, int vdp, int np,
                                  int dtype, void* stream) {
  if (B <= 0 || B > 65535 || T_ <= 0 || heads <= 0 || heads > 65535 || vdp <= 0 || np <= 0 || !decay) return KVB_ERR_ARG;
  kvb::ScanParams p;
  p.dt_bias = p.a_log = p.skip = nullptr; p.decay = decay; p.slots = slots; p.start = start; p.count = count; p.state = state; p.ld = 0;
  p.T = T_; p.dt_col = 0; p.heads = heads; p.groups = heads; p.vdp = vdp; p.np = np; p.inner = heads * vdp; p.channels = 0;
  KVB_SSM_TYPES(dtype, const T* q = (const T*)qk;
                return kvb::scan_simple_launch<T>(nullptr, v, ldv, q + heads * np, q, ldqk, y, p, B, (cudaStream_t)stream));
}

extern "C" int kvb_gated_linear_scan(const kvb_gated_linear* g, const void* v, long long ldv, float* state, void* y, const int* only,
                                     const int* slots, const int* start, const int* count, int B, int T_, int vdp, int dtype, void* stream) {
  if (!g || B <= 0 || B > 65535 || T_ <= 0 || g->heads <= 0 || g->heads > 65535 || vdp <= 0 || g->np <= 0 || g->rank <= 0 ||
      g->ld < 2LL * g->heads * g->np + g->rank)
    return KVB_ERR_ARG;
  kvb::ScanParams p;
  p.dt_bias = p.a_log = p.skip = p.decay = nullptr; p.slots = slots; p.start = start; p.count = count; p.state = state; p.ld = 0;
  p.T = T_; p.dt_col = 0; p.heads = g->heads; p.groups = g->heads; p.vdp = vdp; p.np = g->np; p.inner = g->heads * vdp; p.channels = 0;
  const kvb::RowDecay rd{*g, only};
  KVB_SSM_TYPES(dtype, return (kvb::scan_simple_launch<T, float, true>(nullptr, v, ldv, g->in + g->heads * g->np, g->in, g->ld, y, p, B,
                                                                       (cudaStream_t)stream, rd)));
}

extern "C" int kvb_state_step(const void* u, long long ld, int col, int dt_col, const float* w, const float* bias, const float* dt_bias,
                              const float* a_log, const float* skip, void* ring, float* state, void* y, const int* slots,
                              const int* start, const int* count, int B, int heads, int groups, int vdp, int np, int taps, int dtype,
                              void* stream) {
  if (B <= 0 || B > 65535 || heads <= 0 || groups <= 0 || heads % groups || vdp <= 0 || np <= 0 || taps <= 0) return KVB_ERR_ARG;
  if (vdp % 8 || np % 8) return KVB_ERR_ALIGN;
  if (vdp > 4 * kvb::SS_THREADS) return KVB_ERR_TOO_LARGE;
  const size_t smem = ((size_t)vdp + 2 * np + 4 * kvb::SS_THREADS) * sizeof(float);
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  kvb::StepParams q;
  kvb::ScanParams& p = q.s;
  p.dt_bias = dt_bias; p.a_log = a_log; p.skip = skip; p.decay = nullptr; p.slots = slots; p.start = start; p.count = count;
  p.state = state; p.ld = ld; p.T = 1; p.dt_col = dt_col; p.heads = heads; p.groups = groups; p.vdp = vdp; p.np = np; p.inner = heads * vdp;
  p.channels = heads * vdp + 2 * groups * np;
  q.w = w; q.bias = bias; q.taps = taps; q.col = col;
  KVB_SSM_TYPES(dtype, (kvb::state_step_kernel<T><<<dim3(heads, B), kvb::SS_THREADS, smem, (cudaStream_t)stream>>>(
      (const T*)u, (T*)ring, (T*)y, q)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_gated_group_norm(const void* y, const void* z, long long ld, const float* weight, void* out, long long n, int heads,
                                    int vdim, int vdp, int parts, float eps, int dtype, void* stream) {
  if (n <= 0 || n > 0x7fffffffLL || heads <= 0 || vdim <= 0 || vdp < vdim || parts <= 0 || parts > 65535 || heads * vdim % parts) return KVB_ERR_ARG;
  kvb::GroupNormParams p;
  p.weight = weight; p.ld = ld; p.heads = heads; p.vdim = vdim; p.vdp = vdp; p.size = heads * vdim / parts; p.inner = heads * vdp;
  p.eps = eps;
  KVB_SSM_TYPES(dtype, return kvb::group_norm_launch<T>(y, z, out, p, parts, n, (cudaStream_t)stream));
}

extern "C" int kvb_activate(void* x, long long n, int act, int dtype, void* stream) {
  if (n <= 0 || act != 1) return KVB_ERR_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  const long long per = 256 * (dtype == 0 ? 4 : 8), blocks = (n + per - 1) / per;
  if (blocks > 0x7fffffffLL || (reinterpret_cast<uintptr_t>(x) & 15)) return KVB_ERR_ARG;
  if (dtype == 0) kvb::relu_squared_kernel<float, 4><<<(unsigned)blocks, 256, 0, s>>>((float*)x, n);
  else if (dtype == 1) kvb::relu_squared_kernel<__nv_bfloat16, 8><<<(unsigned)blocks, 256, 0, s>>>((__nv_bfloat16*)x, n);
  else return KVB_ERR_ARG;
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
