// Grouped-query attention over a cache with one row per position, [key (dimp) | value (vdp)] per key/value head.
//
//   prep    root mean squares of the whole query and key projections or of every head, rotation (angles in fp32, once per token),
//           padded queries out, keys and values to their positions in the cache;
//   pool    means of keys and values of the blocks that a pass completes (one token: the end of prep);
//   attend  CUDA cores: fp32, and shapes that the tcgen05 kernel (latent_sm100.cu) does not take;
//   decode  one new token per sequence, bf16: the positions are split over CTAs, K and V tiles come by TMA and meet the heads
//           of a group as mma.sync tiles; a second kernel puts the parts together.
//
// Masks (windows, kept first positions, chunks) are arithmetic: a query has at most two ranges of positions, and only tiles at their
// borders look at single ones. The softmax may have one more term in its denominator (a sink without a value); the output may be
// multiplied with the sigmoid of a gate projection before it is stored. Two maps per head (differential attention) share the values:
// one CTA has both, so that values are read once and the difference and its norm need no pass of their own.
#include <cuda.h>

#include "attn_spec.cuh"
#include "common.cuh"
#include "kvb200_layers.h"
#include "tmap.cuh"

namespace kvb {

// ------------------------------------------------------------------------------------------------ prep
constexpr int GP_THREADS = 128;

template <typename T, int V>
struct alignas(sizeof(T) * V) GpVec {
  T v[V];
};

struct GpParams {
  long long ld;
  const float *norm_q, *norm_k, *freq;
  const int *slots, *start, *count;
  kvb_attention a;
  int T, len, heads, kv_heads, dim, dimp, vdp, rot_dims, value_col;  // heads, kv_heads: of queries and keys, maps counted
  unsigned rot_magic, rest_magic;
};

// Columns [c, c + V) of the sum of the rows first .. last - 1 of block `block` of a sequence; slot: its first row.
template <typename T, int V>
__device__ __forceinline__ void pool_columns(const T* slot, const kvb_attention& a, long long step, int block, int c, int first, int last, float (&s)[V]) {
  using Vec = GpVec<T, V>;
#pragma unroll
  for (int e = 0; e < V; ++e) s[e] = 0.f;
  const int place = row_of(a, block * a.pool);  // a block's rows lie one behind the other up to the end of the ring
  auto add = [&](const T* rows, int j0, int j1) {
#pragma unroll 16
    for (int j = j0; j < j1; ++j) {
      const Vec v = *reinterpret_cast<const Vec*>(rows + (long long)j * step);
#pragma unroll
      for (int e = 0; e < V; ++e) s[e] += to_f32(v.v[e]);
    }
  };
  for (int j0 = 0, at = place; j0 < a.pool; at = a.head) {
    const int n = min(a.pool - j0, a.head + a.ring - at), mid = j0;
    const int lo = max(first, mid), hi = min(last, mid + n);
    if (lo < hi) add(slot + (at - mid) * step + c, lo, hi);
    j0 += n;
  }
}

template <typename T, int V>
__device__ __forceinline__ void pool_store(T* slot, const kvb_attention& a, long long step, int block, int c, const float (&s)[V]) {
  const float inv = 1.f / (float)a.pool;
  GpVec<T, V> r;
#pragma unroll
  for (int e = 0; e < V; ++e) r.v[e] = from_f32<T>(s[e] * inv);
  *reinterpret_cast<GpVec<T, V>*>(slot + block * step + c) = r;
}

// A CTA has a block, a thread V columns of some of its rows.
constexpr int PL_SHARES = 4;

template <typename T, int V>
__global__ void __launch_bounds__(GP_THREADS * PL_SHARES)
grouped_pool_kernel(T* __restrict__ rows, const GpParams p) {
  __shared__ float part[PL_SHARES - 1][GP_THREADS][V + 1];
  const int b = blockIdx.y, block = p.start[b] / p.a.pool + blockIdx.x;
  // complete with this pass, and with a row of its own
  if ((block + 1) * p.a.pool > p.start[b] + p.count[b] || block >= p.a.head) return;
  const int row = p.a.maps * p.a.dimp + p.a.vdp;
  const long long step = (long long)p.a.kv_heads * row;
  T* slot = rows + (long long)p.slots[b] * p.len * step;
  const int lane = threadIdx.x % GP_THREADS, share = threadIdx.x / GP_THREADS, per = (p.a.pool + PL_SHARES - 1) / PL_SHARES;
  for (int c0 = 0; c0 < step; c0 += GP_THREADS * V) {
    const int c = c0 + lane * V;
    float s[V];
    if (c < step) pool_columns<T, V>(slot, p.a, step, block, c, share * per, min(p.a.pool, (share + 1) * per), s);
    if (share > 0 && c < step) {
#pragma unroll
      for (int e = 0; e < V; ++e) part[share - 1][lane][e] = s[e];
    }
    __syncthreads();
    if (share == 0 && c < step) {
#pragma unroll
      for (int k = 0; k < PL_SHARES - 1; ++k)
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] += part[k][lane][e];
      pool_store<T, V>(slot, p.a, step, block, c, s);
    }
    __syncthreads();
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(GP_THREADS)
grouped_prep_kernel(const T* __restrict__ qkv, T* __restrict__ q, T* __restrict__ rows, const GpParams p) {
  using Vec = GpVec<T, V>;
  extern __shared__ float cs_sm[];  // cos | sin, rot_dims / 2 each; with head_norm the factors of all heads
  __shared__ float red[2][GP_THREADS / 32];
  const int t = blockIdx.x, b = blockIdx.y;
  const int half = p.rot_dims / 2, pos = p.start[b] + t;
  const long long n = (long long)b * p.T + t;
  const T* src = qkv + n * p.ld;
  const int nq = p.heads * p.dimp, nk = p.kv_heads * p.dimp;
  for (int k = threadIdx.x; k < half; k += GP_THREADS) sincosf((float)pos * p.freq[k], &cs_sm[half + k], &cs_sm[k]);
  const int maps = p.a.maps, row = maps * p.dimp + p.vdp, place = row_of(p.a, pos);
  // where the token's keys and values go; padding goes nowhere
  T* const dst = (!p.a.borrowed && t < p.count[b] && place < p.len) ? rows + ((long long)p.slots[b] * p.len + place) * p.a.kv_heads * row : nullptr;
  const bool shared = p.value_col == nq;
  // a single token may complete a block; the rows before it are those of earlier passes
  auto pool = [&]() {
    const int size = p.a.pool;
    if (size == 0 || p.T > 1 || !dst || (pos + 1) % size || pos / size >= p.a.head) return;  // the same for all threads
    __syncthreads();
    const long long step = (long long)p.a.kv_heads * row;
    T* slot = rows + (long long)p.slots[b] * p.len * step;
    for (int c = threadIdx.x * V; c < step; c += GP_THREADS * V) {
      float s[V];
      pool_columns<T, V>(slot, p.a, step, pos / size, c, 0, size, s);
      pool_store<T, V>(slot, p.a, step, pos / size, c, s);
    }
  };
  // one piece of a head: the key part of the cache or the query
  auto put = [&](int h, int col, const Vec& v) {
    if (h < p.heads) *reinterpret_cast<Vec*>(q + (n * p.heads + h) * p.dimp + col) = v;
    else if (dst) {
      const int k = h - p.heads, g = maps == 1 ? k : k / maps;
      *reinterpret_cast<Vec*>(dst + g * row + (k - g * maps) * p.dimp + col) = v;
    }
  };
  auto put_values = [&]() {
    for (int i = threadIdx.x * V; i < p.a.kv_heads * p.vdp; i += GP_THREADS * V) {
      const int g = i / p.vdp;
      *reinterpret_cast<Vec*>(dst + g * row + maps * p.dimp + i - g * p.vdp) = *reinterpret_cast<const Vec*>(src + p.value_col + i);
    }
  };
  const int per_head = p.dimp / V;
  const int partner = half / V;  // lanes from one half of a pair to the other
  if (p.norm_q && p.a.head_norm && partner * V == half && (partner & (partner - 1)) == 0 && !shared && per_head <= 32 && (per_head & (per_head - 1)) == 0) {
    // a head lies in neighbouring lanes: one pass, in which pairs of the rotation find each other by a shuffle
    if (dst) put_values();
    if (half > 0) __syncthreads();
    const int total = (nq + nk) / V;
#pragma unroll 4
    for (int i0 = 0; i0 < total; i0 += GP_THREADS) {
      const int i = i0 + threadIdx.x;
      Vec a;
      float s = 0.f;
      if (i < total) {
        a = *reinterpret_cast<const Vec*>(src + i * V);
#pragma unroll
        for (int e = 0; e < V; ++e) s = fmaf(to_f32(a.v[e]), to_f32(a.v[e]), s);
      }
      for (int o = per_head >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      const bool in = i < total;
      const float r = 1.f / sqrtf(s / (float)p.dim + p.a.eps);
      const int h = in ? i / per_head : 0, col = (i - h * per_head) * V;
      float x[V] = {};
      if (in) {
        const float* w = (h < p.heads ? p.norm_q : p.norm_k) + col;
        const float f = p.a.q_scale && h < p.heads ? r * p.a.q_scale[h / maps] : r;
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = to_f32(a.v[e]) * f * w[e];
      }
      if (half > 0) {
        const bool upper = col >= half, rotated = in && col < 2 * half;
        const float* cs = cs_sm + (upper ? col - half : col);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const float y = __shfl_xor_sync(0xffffffffu, x[e], partner);
          if (rotated) x[e] = x[e] * cs[e] + (upper ? y : -y) * cs[half + e];
        }
      }
      if (!in) continue;
#pragma unroll
      for (int e = 0; e < V; ++e) a.v[e] = from_f32<T>(x[e]);
      put(h, col, a);
    }
    pool();
    return;
  }
  float rq = 1.f, rk = 1.f;
  const bool whole = p.norm_q && !p.a.head_norm;
  float* const head_r = cs_sm + p.rot_dims;
  if (p.norm_q && p.a.head_norm) {
    for (int h = threadIdx.x >> 5; h < p.heads + p.kv_heads; h += GP_THREADS / 32) {
      float s = 0.f;
      for (int i = (threadIdx.x & 31) * V; i < p.dimp; i += 32 * V) {
        const Vec a = *reinterpret_cast<const Vec*>(src + h * p.dimp + i);
#pragma unroll
        for (int e = 0; e < V; ++e) s = fmaf(to_f32(a.v[e]), to_f32(a.v[e]), s);
      }
      s = warp_sum(s);
      if ((threadIdx.x & 31) == 0) head_r[h] = 1.f / sqrtf(s / (float)p.dim + p.a.eps);
    }
  }
  if (whole) {
    float ss[2] = {0.f, 0.f};
    for (int i = threadIdx.x * V; i < nq + nk; i += GP_THREADS * V) {
      const Vec a = *reinterpret_cast<const Vec*>(src + i);
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < V; ++e) s = fmaf(to_f32(a.v[e]), to_f32(a.v[e]), s);
      if (i < nq) ss[0] += s;
      else ss[1] += s;
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      ss[u] = warp_sum(ss[u]);
      if ((threadIdx.x & 31) == 0) red[u][threadIdx.x >> 5] = ss[u];
    }
  }
  __syncthreads();
  if (whole) {
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int i = 0; i < GP_THREADS / 32; ++i) {
      s0 += red[0][i];
      s1 += red[1][i];
    }
    rq = 1.f / sqrtf(s0 / (float)(p.heads * p.dim) + p.a.eps);  // padding adds nothing to the sums
    rk = 1.f / sqrtf(s1 / (float)(p.kv_heads * p.dim) + p.a.eps);
  }
  auto normed = [&](int h, int col, const Vec& a, float (&x)[V]) {
    float r = p.norm_q && !whole ? head_r[h] : (h < p.heads ? rq : rk);
    if (p.a.q_scale && h < p.heads) r *= p.a.q_scale[h / maps];
    const float* w = p.norm_q ? (h < p.heads ? p.norm_q + (whole ? h * p.dimp : 0) : p.norm_k + (whole ? (h - p.heads) * p.dimp : 0)) + col : nullptr;
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = p.norm_q ? to_f32(a.v[e]) * r * w[e] : to_f32(a.v[e]) * r;
  };
  const int all = p.heads + p.kv_heads;
  const int ru = half / V;
  for (int i = threadIdx.x; i < all * ru; i += GP_THREADS) {
    const int h = ru == 1 ? i : (int)__umulhi((unsigned)i, p.rot_magic), k = (i - h * ru) * V;
    Vec a = *reinterpret_cast<const Vec*>(src + h * p.dimp + k), c = *reinterpret_cast<const Vec*>(src + h * p.dimp + half + k);
    if (shared && h >= p.heads && dst) {
      T* v = dst + (h - p.heads) * row + p.dimp;
      *reinterpret_cast<Vec*>(v + k) = a;
      *reinterpret_cast<Vec*>(v + half + k) = c;
    }
    float x[V], y[V];
    normed(h, k, a, x);
    normed(h, half + k, c, y);
    const float *cs = cs_sm + k, *sn = cs_sm + half + k;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      a.v[e] = from_f32<T>(x[e] * cs[e] - y[e] * sn[e]);
      c.v[e] = from_f32<T>(y[e] * cs[e] + x[e] * sn[e]);
    }
    put(h, k, a);
    put(h, half + k, c);
  }
  // columns that are not rotated, padding included
  const int re = (p.dimp - p.rot_dims) / V;
  for (int i = threadIdx.x; i < all * re; i += GP_THREADS) {
    const int h = re == 1 ? i : (int)__umulhi((unsigned)i, p.rest_magic), k = p.rot_dims + (i - h * re) * V;
    Vec a = *reinterpret_cast<const Vec*>(src + h * p.dimp + k);
    if (shared && h >= p.heads && dst) *reinterpret_cast<Vec*>(dst + (h - p.heads) * row + p.dimp + k) = a;
    float x[V];
    normed(h, k, a, x);
#pragma unroll
    for (int e = 0; e < V; ++e) a.v[e] = from_f32<T>(x[e]);
    put(h, k, a);
  }
  if (!shared && dst) put_values();
  pool();
}

template <typename T, int V>
static int gp_launch_vec(const void* qkv, void* q, void* rows, GpParams& p, int B, cudaStream_t s) {
  // i / n as a high product, exact for i, n < 2^16
  auto magic = [](int n) { return n > 1 ? (unsigned)(0x100000000ull / n + 1) : 0u; };
  p.rot_magic = magic(p.rot_dims / 2 / V);
  p.rest_magic = magic((p.dimp - p.rot_dims) / V);
  if ((long long)(p.heads + p.kv_heads) * p.dimp >= 65536) return KVB_ERR_TOO_LARGE;
  const size_t smem = (size_t)(p.rot_dims + (p.a.head_norm ? p.heads + p.kv_heads : 0)) * sizeof(float) + 8;
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  grouped_prep_kernel<T, V><<<dim3(p.T, B), GP_THREADS, smem, s>>>((const T*)qkv, (T*)q, (T*)rows, p);
  if (p.a.pool > 0 && p.T > 1) grouped_pool_kernel<T, 16 / sizeof(T)><<<dim3(p.T / p.a.pool + 1, B), GP_THREADS * PL_SHARES, 0, s>>>((T*)rows, p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <typename T>
static int gp_launch(const void* qkv, void* q, void* rows, GpParams& p, int B, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  if ((p.rot_dims / 2) % V == 0 && p.ld % V == 0) return gp_launch_vec<T, V>(qkv, q, rows, p, B, s);
  return gp_launch_vec<T, 1>(qkv, q, rows, p, B, s);
}

// ------------------------------------------------------------------------- attention on CUDA cores
constexpr int GA_WARPS = 4;
constexpr int GA_MAX_V = 16;  // value features per lane

struct GaParams {
  kvb_attention a;
  const int *slots, *start;
  long long gate_ld;
  int T, len;
};

__device__ __forceinline__ float gate_of(float g) { return 1.f / (1.f + expf(-g)); }

// A warp has one head of one query, with all its maps.
template <typename T, int MAPS>
__global__ void __launch_bounds__(GA_WARPS * 32)
grouped_attend_simple_kernel(const T* __restrict__ q, const T* __restrict__ rows, const T* __restrict__ gate, T* __restrict__ out,
                             const GaParams p) {
  extern __shared__ float gq_all[];
  const kvb_attention& a = p.a;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * GA_WARPS + warp, h = blockIdx.y, b = blockIdx.z;
  if (t >= p.T) return;
  const int row = MAPS * a.dimp + a.vdp, g = h / (a.heads / a.kv_heads);
  const long long n = (long long)b * p.T + t, step = (long long)a.kv_heads * row;
  float* qs = gq_all + warp * a.dimp;
  const T* base = rows + (long long)p.slots[b] * p.len * step + (long long)g * row;
  const int hi = a.ring ? p.start[b] + t : min(p.start[b] + t, p.len - 1);  // rows of padding may lie beyond the cache
  const int lo = seen_from(a, hi), kept = a.pool ? blocks_seen(a, hi) : min(a.keep, lo), seen = kept + hi - lo + 1;
  const float sink = a.sink ? (a.sink_w ? a.sink_w[h] : 0.f) : -INFINITY;
  float acc[MAPS][GA_MAX_V];
#pragma unroll
  for (int u = 0; u < MAPS; ++u) {
    __syncwarp();
    for (int i = lane; i < a.dimp; i += 32) qs[i] = to_f32(q[((n * a.heads + h) * MAPS + u) * a.dimp + i]);
    __syncwarp();
    float m = sink, l = a.sink ? 1.f : 0.f;
#pragma unroll
    for (int i = 0; i < GA_MAX_V; ++i) acc[u][i] = 0.f;
    for (int j0 = 0; j0 < seen; j0 += 32) {
      const int j = j0 + lane;
      int place = 0;
      float s = -INFINITY;
      if (j < seen) {
        place = a.pool && j < kept ? j : row_of(a, j < kept ? j : lo + j - kept);
        const T* k = base + place * step + u * a.dimp;
        float a0 = 0.f, a1 = 0.f;
        for (int i = 0; i < a.dimp; i += 2) {
          a0 = fmaf(qs[i], to_f32(k[i]), a0);
          a1 = fmaf(qs[i + 1], to_f32(k[i + 1]), a1);
        }
        s = (a0 + a1) * a.scale;
        if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
      }
      const float mn = fmaxf(m, warp_max(s));
      const float f = expf(m - mn);
      const float w = expf(s - mn);
      m = mn;
      l = fmaf(l, f, warp_sum(w));
#pragma unroll
      for (int i = 0; i < GA_MAX_V; ++i) acc[u][i] *= f;
      const int nk = min(32, seen - j0);
      for (int e = 0; e < nk; ++e) {
        const float we = __shfl_sync(0xffffffffu, w, e);
        const T* v = base + __shfl_sync(0xffffffffu, place, e) * step + MAPS * a.dimp;
#pragma unroll
        for (int i = 0; i < GA_MAX_V; ++i) {
          const int c = i * 32 + lane;
          if (c < a.vdp) acc[u][i] = fmaf(we, to_f32(v[c]), acc[u][i]);
        }
      }
    }
    const float inv = 1.f / l;
#pragma unroll
    for (int i = 0; i < GA_MAX_V; ++i) acc[u][i] *= inv;
  }
  float post = a.post;
  if (MAPS == 2) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < GA_MAX_V; ++i) {
      acc[0][i] = fmaf(-a.lambda, acc[MAPS - 1][i], acc[0][i]);  // zero in the padding
      ss = fmaf(acc[0][i], acc[0][i], ss);
    }
    post = a.post / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
  }
#pragma unroll
  for (int i = 0; i < GA_MAX_V; ++i) {
    const int c = i * 32 + lane;
    if (c >= a.vdp) continue;
    float y = acc[0][i] * post;
    if (gate) y *= gate_of(to_f32(gate[n * p.gate_ld + (a.gate_cols == 1 ? h : h * a.vdp + c)]));
    out[n * a.out_ld + h * a.vdp + c] = from_f32<T>(y);
  }
}

template <typename T>
static int ga_launch(const void* q, const void* rows, const void* gate, void* out, const GaParams& p, int B, cudaStream_t s) {
  const size_t smem = GA_WARPS * p.a.dimp * sizeof(float);
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  const dim3 grid((p.T + GA_WARPS - 1) / GA_WARPS, p.a.heads, B);
  if (p.a.maps == 2) grouped_attend_simple_kernel<T, 2><<<grid, GA_WARPS * 32, smem, s>>>((const T*)q, (const T*)rows, (const T*)gate, (T*)out, p);
  else grouped_attend_simple_kernel<T, 1><<<grid, GA_WARPS * 32, smem, s>>>((const T*)q, (const T*)rows, (const T*)gate, (T*)out, p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

// ------------------------------------------------------------------ single token, bf16 on mma.sync, split over the positions
// A CTA has up to 16 query heads of one key/value head of one sequence and a range of its positions. A warp of its own feeds
// tiles of 64 positions (TMA, 128B-swizzled chunks of 64 columns) into a ring of stages; four warps take 16 positions of
// every tile each. 16 heads x 16 positions is far below a tcgen05 tile. With two maps the 16 rows are 8 heads x 2: the first 8 rows meet
// the first keys, the others the second ones (the other rows of the A operand are zero), and both meet the values at once.
constexpr int GD_WARPS = 4;
constexpr int GD_KEYS = 64;   // positions of a tile
constexpr int GD_HEADS = 16;
constexpr int GD_MAX_SPLIT = 64;
constexpr int GD_MAX_STAGES = 4;
constexpr int GD_CHUNK = GD_KEYS * 128;  // bytes of [64 rows x 64 columns]

struct GdParams {
  const __nv_bfloat16 *q, *gate;
  __nv_bfloat16* out;  // (B, out_ld)
  float* part_o;       // (n_split, B, heads · maps, vdp)
  float* part_ml;      // (n_split, B, heads · maps, 2)
  const int *slots, *start;
  int* status;
  long long gate_ld;
  kvb_attention a;
  int B, len, heads, kv_heads, dimp, vdp, n_split, stages;
  float scale_log2, cap_in, cap_out;  // cap_out > 0: the score in log2 units is cap_out · tanh(cap_in · q·k)
};

__device__ __forceinline__ float gd_sink(const GdParams& p, int h) { return p.a.sink_w ? p.a.sink_w[h] * ATTN_LOG2E : 0.f; }
__device__ __forceinline__ float2 gd_gate(const GdParams& p, int b, int h, int c) {
  const __nv_bfloat16* g = p.gate + b * p.gate_ld;
  if (p.a.gate_cols == 1) {
    const float v = gate_of(__bfloat162float(g[h]));
    return make_float2(v, v);
  }
  const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(g + h * p.vdp + c));
  return make_float2(gate_of(v.x), gate_of(v.y));
}

__device__ __forceinline__ void gd_ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void gd_ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void gd_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// KC, VC: chunks of 64 key and value columns (columns beyond the sizes are zero)
template <int KC, int VC, int MAPS>
__global__ void __launch_bounds__(GD_WARPS * 32 + 32)
grouped_decode_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmK2, const __grid_constant__ CUtensorMap tmV,
                      const GdParams p) {
  extern __shared__ __align__(1024) uint8_t gd_smem[];
  __shared__ float s_ml[GD_WARPS][GD_HEADS][2];
  __shared__ uint64_t full[GD_MAX_STAGES], empty[GD_MAX_STAGES];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  constexpr int STAGE = (KC * MAPS + VC) * GD_CHUNK, HEADS = GD_HEADS / MAPS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int group = p.heads / p.kv_heads, tiles_h = (group + HEADS - 1) / HEADS;
  const int split = blockIdx.x, g = blockIdx.y / tiles_h, b = blockIdx.z;
  const int h0 = g * group + blockIdx.y % tiles_h * HEADS, h_end = min(h0 + HEADS, (g + 1) * group);
  const int hi = p.a.ring ? p.start[b] : min(p.start[b], p.len - 1);
  const int lo = seen_from(p.a, hi), first = lo / GD_KEYS, keep = p.a.keep;
  // tiles of kept positions or of blocks, then those of [lo, hi]
  const int blocks = blocks_seen(p.a, hi);
  const int kept = p.a.pool ? (blocks + GD_KEYS - 1) / GD_KEYS : min((keep + GD_KEYS - 1) / GD_KEYS, first);
  const int nT = kept + hi / GD_KEYS - first + 1;
  auto tile_at = [&](int t) { return t < kept ? t : t - kept + first; };
  const int per = (nT + p.n_split - 1) / p.n_split;
  const int ta = split * per, tb = min(nT, ta + per);
  if (smem_u32(gd_smem) & 1023u) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, STATUS_TIMEOUT_MISC);
    return;
  }
  if (threadIdx.x == 0) {
    for (int i = 0; i < GD_MAX_STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], GD_WARPS);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  __syncthreads();
  if (warp == GD_WARPS) {
    // ------------------------------------------------------------ producer
    if (lane == 0) {
      tma_prefetch_desc(&tmK);
      if (MAPS == 2) tma_prefetch_desc(&tmK2);
      tma_prefetch_desc(&tmV);
      const int slot = p.slots[b];
      bool ok = true;
      int st = 0;
      uint32_t ph = 0;
      for (int t = ta; t < tb; ++t) {
        if (!(ok = mbar_wait_bounded(&empty[st], ph ^ 1, abort_flag, p.status, STATUS_TIMEOUT_EMPTY))) break;
        mbar_expect_tx(&full[st], (uint32_t)STAGE);
        uint8_t* d = gd_smem + st * STAGE;
        const int row = p.a.pool && t < kept ? t * GD_KEYS : row_of(p.a, tile_at(t) * GD_KEYS);
        for (int c = 0; c < KC; ++c) tma_load_4d(d + c * GD_CHUNK, &tmK, &full[st], 64 * c, g, row, slot);
        if (MAPS == 2)
          for (int c = 0; c < KC; ++c) tma_load_4d(d + (KC + c) * GD_CHUNK, &tmK2, &full[st], 64 * c, g, row, slot);
        for (int c = 0; c < VC; ++c) tma_load_4d(d + (KC * MAPS + c) * GD_CHUNK, &tmV, &full[st], 64 * c, g, row, slot);
        if (++st == p.stages) {
          st = 0;
          ph ^= 1;
        }
      }
      if (!ok) {  // copies in flight get a bounded time to land before the shared memory is released
        const long long c0 = clock64();
        while (clock64() - c0 < 2000000LL) {
        }
      }
    }
    __syncwarp();
    // the barriers of the merge
    for (int i = 0; i < GD_WARPS + 1; ++i) __syncthreads();
    return;
  }
  // queries as A operands: rows lane / 4 and + 8, columns (lane % 4) · 2 and + 8 of a step; zero beyond heads and columns
  uint32_t qf[4 * KC][4];
#pragma unroll
  for (int i = 0; i < 4 * KC; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = h0 + (lane >> 2) + (MAPS == 2 ? 0 : 8 * (e & 1)), c = i * 16 + (lane & 3) * 2 + 8 * (e >> 1);
      qf[i][e] = 0u;
      if (h < h_end && c < p.dimp)
        qf[i][e] = *reinterpret_cast<const uint32_t*>(p.q + (((long long)b * p.heads + h) * MAPS + (MAPS == 2 ? e & 1 : 0)) * p.dimp + c);
    }
  float acc[8 * VC][4];
#pragma unroll
  for (int j = 0; j < 8 * VC; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};  // of heads lane / 4 and + 8; sums of this lane's positions
  // ldmatrix offsets of the four 16-column steps of a chunk: rows = positions, for the values transposed
  uint32_t koff[4], voff[4];
  {
    const int kr = warp * 16 + (lane & 7) + ((lane >> 4) << 3), vr = warp * 16 + (lane & 15);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      koff[i] = (uint32_t)(kr * 128 + (((i * 2 + ((lane >> 3) & 1)) ^ (kr & 7)) << 4));
      voff[i] = (uint32_t)(KC * MAPS * GD_CHUNK + vr * 128 + (((i * 2 + (lane >> 4)) ^ (vr & 7)) << 4));
    }
  }
  bool ok = true;
  int st = 0;
  uint32_t ph = 0;
#pragma unroll 1
  for (int t = ta; t < tb; ++t) {
    // after a wait that ran out the tiles are worked on unseen: the status word tells, and the loop ends
    if (ok) ok = mbar_wait_bounded(&full[st], ph, abort_flag, p.status, STATUS_TIMEOUT_FULL);
    const uint32_t tile = smem_u32(gd_smem) + (uint32_t)(st * STAGE);
    const int jw = tile_at(t) * GD_KEYS + warp * 16;  // this warp's 16 positions, or blocks
    const bool of_blocks = p.a.pool && t < kept;
    const int first_j = of_blocks ? 0 : lo, last_j = of_blocks ? blocks - 1 : hi;
    if (jw <= last_j && (jw + 15 >= first_j || jw < keep)) {
      float s[2][2][4];  // even and odd steps apart: two short chains instead of a long one
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[0][n][e] = s[1][n][e] = 0.f;
#pragma unroll
      for (int k = 0; k < 4 * KC; ++k) {
        uint32_t bb[4];
        gd_ldsm4(bb, tile + (uint32_t)((k >> 2) * GD_CHUNK) + koff[k & 3]);
        if (MAPS == 1) {
          gd_mma(s[k & 1][0], qf[k], bb[0], bb[1]);
          gd_mma(s[k & 1][1], qf[k], bb[2], bb[3]);
        } else {
          const uint32_t qa[4] = {qf[k][0], 0u, qf[k][2], 0u}, qb[4] = {0u, qf[k][1], 0u, qf[k][3]};
          gd_mma(s[k & 1][0], qa, bb[0], bb[1]);
          gd_mma(s[k & 1][1], qa, bb[2], bb[3]);
          gd_ldsm4(bb, tile + (uint32_t)((KC + (k >> 2)) * GD_CHUNK) + koff[k & 3]);
          gd_mma(s[k & 1][0], qb, bb[0], bb[1]);
          gd_mma(s[k & 1][1], qb, bb[2], bb[3]);
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[0][n][e] = (s[0][n][e] + s[1][n][e]) * p.scale_log2;
      if (p.cap_out > 0.f) {  // scale_log2 is cap_in then
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[0][n][e] = p.cap_out * cap_tanh(s[0][n][e]);
      }
      if (jw + 15 > last_j || (jw < first_j && jw + 15 >= keep)) {
        const int j0 = jw + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int j = j0 + 8 * n + (e & 1);
            if (j > last_j || (j < first_j && j >= keep)) s[0][n][e] = -INFINITY;
          }
      }
      float f[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float m = fmaxf(fmaxf(s[0][0][2 * r], s[0][0][2 * r + 1]), fmaxf(s[0][1][2 * r], s[0][1][2 * r + 1]));
        m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
        m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
        m = fmaxf(m, mx[r]);
        f[r] = attn_exp2(mx[r] - m);
        mx[r] = m;
        float w = 0.f;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 2 * r; e < 2 * r + 2; ++e) {
            s[0][n][e] = attn_exp2(s[0][n][e] - m);
            w += s[0][n][e];
          }
        sum[r] = fmaf(sum[r], f[r], w);
      }
      if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
        for (int j = 0; j < 8 * VC; ++j) {
          acc[j][0] *= f[0];
          acc[j][1] *= f[0];
          acc[j][2] *= f[1];
          acc[j][3] *= f[1];
        }
      }
      const uint32_t pa[4] = {pack_bf16x2(s[0][0][0], s[0][0][1]), pack_bf16x2(s[0][0][2], s[0][0][3]),
                              pack_bf16x2(s[0][1][0], s[0][1][1]), pack_bf16x2(s[0][1][2], s[0][1][3])};
#pragma unroll
      for (int j = 0; j < 4 * VC; ++j) {
        uint32_t v[4];
        gd_ldsm4t(v, tile + (uint32_t)((j >> 2) * GD_CHUNK) + voff[j & 3]);
        gd_mma(acc[2 * j], pa, v[0], v[1]);
        gd_mma(acc[2 * j + 1], pa, v[2], v[3]);
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st]);
    if (++st == p.stages) {
      st = 0;
      ph ^= 1;
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
    sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
    if ((lane & 3) == 0) {
      s_ml[warp][(lane >> 2) + 8 * r][0] = mx[r];
      s_ml[warp][(lane >> 2) + 8 * r][1] = sum[r];
    }
  }
  __syncthreads();  // nobody reads the stages any more
  float* so = reinterpret_cast<float*>(gd_smem);  // (GD_HEADS, vdp), filled warp by warp
  for (int w = 0; w < GD_WARPS; ++w) {
    if (w == warp) {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int hr = (lane >> 2) + 8 * r;
        float m = -INFINITY;
#pragma unroll
        for (int k = 0; k < GD_WARPS; ++k) m = fmaxf(m, s_ml[k][hr][0]);
        const float f = mx[r] == -INFINITY ? 0.f : attn_exp2(mx[r] - m);
#pragma unroll
        for (int j = 0; j < 8 * VC; ++j) {
          const int c = j * 8 + (lane & 3) * 2;
          if (c >= p.vdp) continue;
          float2* d = reinterpret_cast<float2*>(so + hr * p.vdp + c);
          float2 v = w == 0 ? make_float2(0.f, 0.f) : *d;
          v.x = fmaf(f, acc[j][2 * r], v.x);
          v.y = fmaf(f, acc[j][2 * r + 1], v.y);
          *d = v;
        }
      }
    }
    __syncthreads();
  }
  // the whole softmax of a row: its maximum and sum
  auto totals = [&](int hr, float& m, float& l) {
    m = -INFINITY;
    l = 0.f;
#pragma unroll
    for (int k = 0; k < GD_WARPS; ++k) m = fmaxf(m, s_ml[k][hr][0]);
#pragma unroll
    for (int k = 0; k < GD_WARPS; ++k) l += s_ml[k][hr][0] == -INFINITY ? 0.f : s_ml[k][hr][1] * attn_exp2(s_ml[k][hr][0] - m);
  };
  for (int e = warp; e < h_end - h0; e += GD_WARPS) {
    const int h = h0 + e;
    float m[MAPS], l[MAPS];
#pragma unroll
    for (int u = 0; u < MAPS; ++u) totals(e + 8 * u, m[u], l[u]);
    if (p.n_split > 1) {
#pragma unroll
      for (int u = 0; u < MAPS; ++u) {
        const long long part = ((long long)split * p.B + b) * p.heads * MAPS + h * MAPS + u;
        if (lane == 0) *reinterpret_cast<float2*>(p.part_ml + part * 2) = make_float2(m[u], l[u]);
        for (int c = lane * 4; c < p.vdp; c += 128)
          *reinterpret_cast<float4*>(p.part_o + part * p.vdp + c) = *reinterpret_cast<const float4*>(so + (e + 8 * u) * p.vdp + c);
      }
      continue;
    }
    __nv_bfloat16* dst = p.out + b * p.a.out_ld + h * p.vdp;
    if (MAPS == 2) {
      const float f0 = 1.f / l[0], f1 = p.a.lambda / l[MAPS - 1];
      float ss = 0.f;
      auto diff = [&](int c) {
        const float2 x = *reinterpret_cast<const float2*>(so + e * p.vdp + c), y = *reinterpret_cast<const float2*>(so + (e + 8) * p.vdp + c);
        return make_float2(x.x * f0 - y.x * f1, x.y * f0 - y.y * f1);
      };
      for (int c = lane * 2; c < p.vdp; c += 64) {
        const float2 v = diff(c);
        ss += v.x * v.x + v.y * v.y;
      }
      const float r = p.a.post / sqrtf(warp_sum(ss) / (float)p.a.vdim + p.a.eps);
      for (int c = lane * 2; c < p.vdp; c += 64) {
        const float2 v = diff(c);
        *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(v.x * r, v.y * r);
      }
      continue;
    }
    // the sink may lie far above all scores: everything relative to the larger of both
    const float sink = p.a.sink ? gd_sink(p, h) : -INFINITY;
    const float top = fmaxf(m[0], sink);
    const float f = attn_exp2(m[0] - top), inv = p.a.post * f / (l[0] * f + (p.a.sink ? attn_exp2(sink - top) : 0.f));
    for (int c = lane * 2; c < p.vdp; c += 64) {
      float2 v = *reinterpret_cast<const float2*>(so + e * p.vdp + c);
      v.x *= inv;
      v.y *= inv;
      if (p.gate) {
        const float2 gt = gd_gate(p, b, h, c);
        v.x *= gt.x;
        v.y *= gt.y;
      }
      *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(v.x, v.y);
    }
  }
}

template <int MAPS>
__global__ void __launch_bounds__(128)
grouped_merge_kernel(const GdParams p) {
  __shared__ float wt[MAPS][GD_MAX_SPLIT];
  __shared__ float red[4];
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long long bh = ((long long)b * p.heads + h) * MAPS, step = (long long)p.B * p.heads * MAPS;
  if (warp < MAPS) {
    float m[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = lane + 32 * i;
      const float2 v = s < p.n_split ? *reinterpret_cast<const float2*>(p.part_ml + (s * step + bh + warp) * 2) : make_float2(-INFINITY, 0.f);
      m[i] = v.x;
      l[i] = v.y;
    }
    const float sink = p.a.sink ? gd_sink(p, h) : -INFINITY;
    const float top = fmaxf(warp_max(fmaxf(m[0], m[1])), sink);
    float f[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) f[i] = m[i] == -INFINITY ? 0.f : attn_exp2(m[i] - top);
    const float inv = 1.f / (warp_sum(f[0] * l[0] + f[1] * l[1]) + (p.a.sink ? attn_exp2(sink - top) : 0.f));
    const float scale = MAPS == 2 ? inv : inv * p.a.post;
    wt[warp][lane] = f[0] * scale;
    wt[warp][lane + 32] = f[1] * scale;
  }
  __syncthreads();
  const int c = threadIdx.x * 2;  // value sizes up to 256
  float2 o[MAPS];
#pragma unroll
  for (int u = 0; u < MAPS; ++u) {
    o[u] = make_float2(0.f, 0.f);
    if (c >= p.vdp) continue;
#pragma unroll 8
    for (int s = 0; s < p.n_split; ++s) {
      const float2 v = *reinterpret_cast<const float2*>(p.part_o + (s * step + bh + u) * p.vdp + c);
      const float w = wt[u][s];  // 0 for a part that saw no position (its sums are zero)
      o[u].x = fmaf(w, v.x, o[u].x);
      o[u].y = fmaf(w, v.y, o[u].y);
    }
  }
  if (MAPS == 2) {
    o[0].x = fmaf(-p.a.lambda, o[MAPS - 1].x, o[0].x);
    o[0].y = fmaf(-p.a.lambda, o[MAPS - 1].y, o[0].y);
    const float s = warp_sum(o[0].x * o[0].x + o[0].y * o[0].y);
    if (lane == 0) red[warp] = s;
    __syncthreads();
    const float r = p.a.post / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)p.a.vdim + p.a.eps);
    o[0].x *= r;
    o[0].y *= r;
  }
  if (c >= p.vdp) return;
  if (p.gate) {
    const float2 gt = gd_gate(p, b, h, c);
    o[0].x *= gt.x;
    o[0].y *= gt.y;
  }
  *reinterpret_cast<uint32_t*>(p.out + b * p.a.out_ld + h * p.vdp + c) = pack_bf16x2(o[0].x, o[0].y);
}

// chunks of 64 key columns and of 64 value columns that a kernel is compiled for
static void gd_chunks(const kvb_attention& a, int& kc, int& vc) {
  auto up = [](int n) { return n <= 64 ? 1 : n <= 128 ? 2 : 4; };
  kc = up(a.dimp);
  vc = up(a.vdp);
  if (a.maps == 1) kc = vc = kc > vc ? kc : vc;
  else if (vc < kc) vc = kc;  // built: 1 / 1, 1 / 2, 2 / 2, 1 / 4, 2 / 4
}

static int gd_stage_bytes(const kvb_attention& a) {
  int kc, vc;
  gd_chunks(a, kc, vc);
  return (kc * a.maps + vc) * GD_CHUNK;
}

// parts of the positions: full waves of CTAs, but not so many that starting and ending them costs more than it gains
static int gd_split(int B, int len, const kvb_attention& a) {
  const int group = a.heads / a.kv_heads, per = GD_HEADS / a.maps;
  const long long ctas = (long long)B * a.kv_heads * ((group + per - 1) / per);
  long long tiles = (len + GD_KEYS - 1) / GD_KEYS;
  const int span = a.chunk > 0 ? a.chunk : a.window;
  if (span > 0) {
    const long long most = ((a.pool > 0 ? a.head : a.keep) + GD_KEYS - 1) / GD_KEYS + (span + GD_KEYS - 1) / GD_KEYS + 1;
    if (tiles > most) tiles = most;
  }
  const long long slots = 148 * (gd_stage_bytes(a) * 3 > 110 * 1024 ? 1 : 2);
  int best = 1;
  double best_cost = 1e30;
  for (int n = 1; n <= GD_MAX_SPLIT && n <= tiles; ++n) {
    const double waves = (double)((ctas * n + slots - 1) / slots);
    const double cost = waves * ((double)((tiles + n - 1) / n) + 5.0) + (n > 1 ? 4.0 + 0.1 * n : 0.0);
    if (cost < best_cost) {
      best_cost = cost;
      best = n;
    }
  }
  return best;
}

template <int KC, int VC, int MAPS>
static int gd_launch(const CUtensorMap* tm, GdParams& p, cudaStream_t s) {
  constexpr int stage = (KC * MAPS + VC) * GD_CHUNK;
  p.stages = stage * 4 <= 100 * 1024 ? 4 : stage * 3 <= 220 * 1024 ? 3 : 2;
  const size_t smem = (size_t)p.stages * stage;
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(grouped_decode_kernel<KC, VC, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  const int group = p.heads / p.kv_heads, per = GD_HEADS / MAPS;
  const dim3 grid(p.n_split, p.kv_heads * ((group + per - 1) / per), p.B);
  grouped_decode_kernel<KC, VC, MAPS><<<grid, GD_WARPS * 32 + 32, smem, s>>>(tm[0], tm[1], tm[2], p);
  if (p.n_split > 1) grouped_merge_kernel<MAPS><<<dim3(p.heads, p.B), 128, 0, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

// what every entry point asks of a description
static bool attention_valid(const kvb_attention* a) {
  return a && a->heads > 0 && a->kv_heads > 0 && a->heads % a->kv_heads == 0 && (a->maps == 1 || a->maps == 2) && a->dim > 0 && a->vdim > 0 &&
         a->dimp >= a->dim && a->vdp >= a->vdim && a->window >= 0 && a->keep >= 0 && a->chunk >= 0 && !(a->window && a->chunk) &&
         (a->window || !a->keep) && a->head >= 0 && a->ring >= 0 && a->head % 128 == 0 && a->ring % 128 == 0 && (!a->ring || a->head >= a->keep) &&
         a->pool >= 0 && (!a->pool || (a->window > 0 && a->keep == 0 && a->ring > 0)) && a->out_ld >= (long long)a->heads * a->vdp &&
         a->softcap >= 0.f && !(a->maps == 2 && (a->sink || a->gate_cols)) && (a->gate_cols == 0 || a->gate_cols == 1 || a->gate_cols == a->vdp);
}

}  // namespace kvb

#define KVB_GROUPED_TYPES(dtype, ...)                         \
  switch (dtype) {                                            \
    case 0: { using T = float; __VA_ARGS__; break; }          \
    case 1: { using T = __nv_bfloat16; __VA_ARGS__; break; }  \
    default: return KVB_ERR_ARG;                              \
  }

extern "C" int kvb_grouped_prep(const void* qkv, long long ld, const float* norm_q, const float* norm_k, const float* freq, void* q,
                                void* rows, const int* slots, const int* start, const int* count, int B, int T_, int len,
                                const kvb_attention* a, int dtype, void* stream) {
  if (!kvb::attention_valid(a) || B <= 0 || B > 65535 || T_ <= 0 || len <= 0 || a->rot_dims > a->dim || a->rot_dims % 2 ||
      (norm_q == nullptr) != (norm_k == nullptr) || (a->ring && a->head + a->ring > len))
    return KVB_ERR_ARG;
  if ((a->dimp | a->vdp | a->value_col) % 8) return KVB_ERR_ALIGN;
  if (!a->borrowed && a->value_col == a->heads * a->maps * a->dimp && (a->vdp != a->dimp || a->maps != 1)) return KVB_ERR_ARG;
  kvb::GpParams p;
  p.ld = ld; p.norm_q = norm_q; p.norm_k = norm_k; p.freq = freq; p.slots = slots; p.start = start; p.count = count; p.a = *a;
  p.T = T_; p.len = len; p.heads = a->heads * a->maps; p.kv_heads = a->borrowed ? 0 : a->kv_heads * a->maps; p.dim = a->dim; p.dimp = a->dimp; p.vdp = a->vdp;
  p.rot_dims = a->rot_dims; p.value_col = a->value_col;
  KVB_GROUPED_TYPES(dtype, return kvb::gp_launch<T>(qkv, q, rows, p, B, (cudaStream_t)stream));
}

extern "C" int kvb_grouped_attend(const void* q, const void* rows, const void* gate, long long gate_ld, void* out, const int* slots,
                                  const int* start, int B, int T_, int len, const kvb_attention* a, int dtype, void* stream) {
  if (!kvb::attention_valid(a) || B <= 0 || T_ <= 0 || len <= 0 || B > 65535 || a->heads > 65535 || a->dimp % 2 || (a->ring && a->head + a->ring > len))
    return KVB_ERR_ARG;
  if (a->vdp > 32 * kvb::GA_MAX_V) return KVB_ERR_TOO_LARGE;
  kvb::GaParams p;
  p.a = *a; p.slots = slots; p.start = start; p.gate_ld = gate_ld; p.T = T_; p.len = len;
  KVB_GROUPED_TYPES(dtype, return kvb::ga_launch<T>(q, rows, gate, out, p, B, (cudaStream_t)stream));
}

// ------------------------------------------------------------------------------------- single token
extern "C" int kvb_grouped_decode_supported(const kvb_attention* a) {
  return kvb::attention_valid(a) && a->dimp % 8 == 0 && a->vdp % 8 == 0 && a->dimp <= (a->maps == 2 ? 128 : 256) && a->vdp <= 256;
}

extern "C" long long kvb_grouped_decode_scratch_bytes(int B, int len, const kvb_attention* a) {
  const int n = kvb::gd_split(B, len, *a);
  return n > 1 ? (long long)n * B * a->heads * a->maps * (a->vdp + 2) * 4 : 0;
}

extern "C" int kvb_grouped_decode(const void* q, const void* rows, const void* gate, long long gate_ld, void* out, void* scratch,
                                  const int* slots, const int* start, int B, int n_slots, int len, const kvb_attention* a, int* status,
                                  void* stream) {
  using namespace kvb;
  if (!attention_valid(a) || B <= 0 || B > 65535 || n_slots <= 0 || len <= 0 || !(a->scale > 0.f) || (a->ring && a->head + a->ring > len))
    return KVB_ERR_ARG;
  if (!kvb_grouped_decode_supported(a)) return KVB_ERR_UNSUPPORTED;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(rows) | reinterpret_cast<uintptr_t>(out)) & 15) return KVB_ERR_ALIGN;
  if (a->out_ld % 2) return KVB_ERR_ALIGN;
  if (a->gate_cols > 1 && (gate_ld & 1 || reinterpret_cast<uintptr_t>(gate) & 3)) return KVB_ERR_ALIGN;
  const uint64_t row = a->maps * a->dimp + a->vdp, G = a->kv_heads, sk[3] = {row, G * row, (uint64_t)len * G * row};
  const uint64_t dk[4] = {(uint64_t)a->dimp, G, (uint64_t)len, (uint64_t)n_slots}, dv[4] = {(uint64_t)a->vdp, G, (uint64_t)len, (uint64_t)n_slots};
  const uint32_t box[4] = {64, 1, GD_KEYS, 1};
  CUtensorMap tm[3];
  int rc;
  const __nv_bfloat16* kb = (const __nv_bfloat16*)rows;
  if ((rc = tmap_bf16(&tm[0], kb, 4, dk, sk, box))) return rc;
  if ((rc = tmap_bf16(&tm[1], kb + (a->maps - 1) * a->dimp, 4, dk, sk, box))) return rc;
  if ((rc = tmap_bf16(&tm[2], kb + a->maps * a->dimp, 4, dv, sk, box))) return rc;
  GdParams p;
  p.q = (const __nv_bfloat16*)q; p.gate = (const __nv_bfloat16*)gate; p.status = status; p.a = *a;
  p.out = (__nv_bfloat16*)out; p.slots = slots; p.start = start; p.gate_ld = gate_ld; p.B = B; p.len = len; p.heads = a->heads;
  p.kv_heads = a->kv_heads; p.dimp = a->dimp; p.vdp = a->vdp;
  p.cap_in = a->softcap > 0.f ? a->scale / a->softcap : 0.f;
  p.cap_out = a->softcap * ATTN_LOG2E;
  p.scale_log2 = a->softcap > 0.f ? p.cap_in : a->scale * ATTN_LOG2E;
  p.n_split = gd_split(B, len, *a);
  if (p.n_split > 1 && !scratch) return KVB_ERR_ARG;
  p.part_o = (float*)scratch;
  p.part_ml = p.part_o + (long long)p.n_split * B * a->heads * a->maps * a->vdp;
  int kc, vc;
  gd_chunks(*a, kc, vc);
  cudaStream_t s = (cudaStream_t)stream;
  if (a->maps == 2) {
    if (kc == 1) return vc == 1 ? gd_launch<1, 1, 2>(tm, p, s) : vc == 2 ? gd_launch<1, 2, 2>(tm, p, s) : gd_launch<1, 4, 2>(tm, p, s);
    return vc == 2 ? gd_launch<2, 2, 2>(tm, p, s) : gd_launch<2, 4, 2>(tm, p, s);
  }
  if (kc == 1) return gd_launch<1, 1, 1>(tm, p, s);
  if (kc == 2) return gd_launch<2, 2, 1>(tm, p, s);
  return gd_launch<4, 4, 1>(tm, p, s);
}
