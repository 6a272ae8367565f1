// Retention (linear attention with a fixed decay per head): S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t with rotated queries and keys,
// o normed per head and gated. The recurrence over several tokens is the one of state-space mixers (ssm.cu, ssm_sm100.cu); here are
//
//   prep   rotation of the fp32 projections of queries and keys, rounded once to the type of the scan's operands;
//   norm   y / rms(y) · silu(gate), possibly with a weight (gated linear attention), a few lanes per head of a token;
//   step   one new token per sequence: rotation, decay, state, output, norm and gate of a head in one kernel, all in fp32, bound by
//          reading and writing the state once.
#include "common.cuh"
#include "kvb200_layers.h"
#include "ssm.cuh"

namespace kvb {

template <typename T, int V>
struct alignas(sizeof(T) * V) RtVec {
  T v[V];
};

// ------------------------------------------------------------------------------------------------ prep
constexpr int RP_THREADS = 128;

struct RetPrepParams {
  const float* freq;
  const int* start;
  long long ld;
  int T, heads, np, rot_dims;
  float key_scale;
};

template <typename T, int V>
__global__ void __launch_bounds__(RP_THREADS)
retention_prep_kernel(const float* __restrict__ in, T* __restrict__ out, const RetPrepParams p) {
  using In = RtVec<float, V>;
  using Out = RtVec<T, V>;
  extern __shared__ float rt_cs[];  // cos | sin, rot_dims / 2 each
  const int t = blockIdx.x, b = blockIdx.y, half = p.rot_dims / 2, pos = p.start[b] + t;
  const long long n = (long long)b * p.T + t;
  for (int k = threadIdx.x; k < half; k += RP_THREADS) sincosf((float)pos * p.freq[k], &rt_cs[half + k], &rt_cs[k]);
  __syncthreads();
  const float* src = in + n * p.ld;
  T* dst = out + n * 2 * p.heads * p.np;
  const int ru = half / V, re = (p.np - p.rot_dims) / V;
  for (int i = threadIdx.x; i < 2 * p.heads * ru; i += RP_THREADS) {
    const int h = i / ru, k = (i - h * ru) * V;
    const float f = h < p.heads ? 1.f : p.key_scale;
    const In a = *reinterpret_cast<const In*>(src + h * p.np + k), c = *reinterpret_cast<const In*>(src + h * p.np + half + k);
    Out x, y;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float cs = rt_cs[k + e], sn = rt_cs[half + k + e];
      x.v[e] = from_f32<T>((a.v[e] * cs - c.v[e] * sn) * f);
      y.v[e] = from_f32<T>((c.v[e] * cs + a.v[e] * sn) * f);
    }
    *reinterpret_cast<Out*>(dst + h * p.np + k) = x;
    *reinterpret_cast<Out*>(dst + h * p.np + half + k) = y;
  }
  for (int i = threadIdx.x; i < 2 * p.heads * re; i += RP_THREADS) {
    const int h = i / re, k = p.rot_dims + (i - h * re) * V;
    const float f = h < p.heads ? 1.f : p.key_scale;
    const In a = *reinterpret_cast<const In*>(src + h * p.np + k);
    Out x;
#pragma unroll
    for (int e = 0; e < V; ++e) x.v[e] = from_f32<T>(a.v[e] * f);
    *reinterpret_cast<Out*>(dst + h * p.np + k) = x;
  }
}

// ------------------------------------------------------------------------------------------------ norm
constexpr int HN_WARPS = 8;
constexpr int HN_ROWS = 4;  // rows (heads of tokens) that a group of lanes works on side by side
constexpr int HN_MAX = 16;  // accesses per lane and row

struct HeadNormParams {
  const float* weight;  // (vdp), NULL: ones
  long long ld, rows;
  int heads, vdim, vdp;
  float eps;
};

// LANES lanes have a row; NC accesses of V columns per lane.
template <typename T, int V, int LANES, int NC, int ROWS>
__global__ void __launch_bounds__(HN_WARPS * 32)
head_norm_gate_kernel(const T* __restrict__ y, const T* __restrict__ gate, T* __restrict__ out, const HeadNormParams p) {
  using Vec = RtVec<T, V>;
  constexpr int PER = HN_WARPS * 32 / LANES;  // rows that a CTA works on at a time
  const int lane = threadIdx.x % LANES;
  const unsigned r0 = blockIdx.x * (unsigned)(PER * ROWS) + threadIdx.x / LANES, rows = (unsigned)p.rows, heads = (unsigned)p.heads;
  unsigned n = r0 / heads, h = r0 - n * heads;  // token and head
  Vec v[ROWS][NC], z[ROWS][NC];
  float ss[ROWS];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const unsigned r = r0 + i * PER;
    const bool in = r < rows;
    const T* g = gate + n * p.ld + h * (unsigned)p.vdp;
    for (h += PER; h >= heads; h -= heads) ++n;
#pragma unroll
    for (int k = 0; k < NC; ++k) {
      const int c = (k * LANES + lane) * V;
      if (in && c < p.vdp) {
        v[i][k] = *reinterpret_cast<const Vec*>(y + (long long)r * p.vdp + c);
        z[i][k] = *reinterpret_cast<const Vec*>(g + c);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) v[i][k].v[e] = z[i][k].v[e] = from_f32<T>(0.f);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    ss[i] = 0.f;
#pragma unroll
    for (int k = 0; k < NC; ++k)
#pragma unroll
      for (int e = 0; e < V; ++e) ss[i] = fmaf(to_f32(v[i][k].v[e]), to_f32(v[i][k].v[e]), ss[i]);  // padding is zero
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const unsigned r = r0 + i * PER;
    if (r >= rows) break;
    const float f = 1.f / sqrtf(ss[i] / (float)p.vdim + p.eps);
#pragma unroll
    for (int k = 0; k < NC; ++k) {
      const int c = (k * LANES + lane) * V;
      if (c >= p.vdp) break;
      Vec o;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float w = p.weight ? f * p.weight[c + e] : f;
        o.v[e] = from_f32<T>(to_f32(v[i][k].v[e]) * w * ss_silu_for<T>(to_f32(z[i][k].v[e])));
      }
      *reinterpret_cast<Vec*>(out + (long long)r * p.vdp + c) = o;
    }
  }
}

template <typename T, int V, int LANES, int NC, int ROWS>
static int hn_launch(const void* y, const void* gate, void* out, const HeadNormParams& p, cudaStream_t s) {
  constexpr int per = HN_WARPS * 32 / LANES * ROWS;
  const long long blocks = (p.rows + per - 1) / per;
  if (blocks > 0x7fffffffLL) return KVB_ERR_TOO_LARGE;
  head_norm_gate_kernel<T, V, LANES, NC, ROWS><<<(unsigned)blocks, HN_WARPS * 32, 0, s>>>((const T*)y, (const T*)gate, (T*)out, p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <typename T>
static int hn_type(const void* y, const void* gate, void* out, const HeadNormParams& p, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  if (p.vdp <= 8 * V) return hn_launch<T, V, 8, 1, HN_ROWS>(y, gate, out, p, s);
  if (p.vdp <= 16 * V) return hn_launch<T, V, 16, 1, HN_ROWS>(y, gate, out, p, s);
  if (p.vdp <= 32 * V) return hn_launch<T, V, 32, 1, HN_ROWS>(y, gate, out, p, s);
  if (p.vdp <= 64 * V) return hn_launch<T, V, 32, 2, 2>(y, gate, out, p, s);
  if (p.vdp <= 32 * V * HN_MAX) return hn_launch<T, V, 32, HN_MAX, 1>(y, gate, out, p, s);
  return KVB_ERR_TOO_LARGE;
}

// ------------------------------------------------------------------------------------------------ step
constexpr int RS_THREADS = 256;
constexpr int RS_BATCH = 8;  // float4 of the state that a thread has in flight

struct RetStepParams {
  const float *freq, *decay;
  const int *slots, *start, *count;
  float* state;
  long long ld;
  int heads, vdim, vdp, np, rot_dims;
  float key_scale, eps;
};

// One head of one sequence. Thread (row, quad) has four value columns of rows row, row + n_rows, ...
template <typename T>
__global__ void __launch_bounds__(RS_THREADS)
retention_step_kernel(const float* __restrict__ u, T* __restrict__ out, const RetStepParams p) {
  extern __shared__ float rs_sm[];  // q (np) | k (np) | v (vdp) | partial sums (RS_THREADS · 4)
  __shared__ float red[RS_THREADS / 32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  T* yr = out + ((long long)b * p.heads + h) * p.vdp;
  if (p.count[b] <= 0) {
    for (int i = tid; i < p.vdp; i += RS_THREADS) yr[i] = from_f32<T>(0.f);
    return;
  }
  float *sq = rs_sm, *sk = sq + p.np, *sv = sk + p.np, *part = sv + p.vdp;
  const int quads = p.vdp / 4, n_rows = RS_THREADS / quads;
  const int row0 = tid / quads, quad = tid - row0 * quads;
  const bool active = row0 < n_rows;
  const int start = p.start[b];
  float4* st = reinterpret_cast<float4*>(p.state + ((long long)p.slots[b] * p.heads + h) * p.np * p.vdp) + quad;
  float4 s[RS_BATCH];
  auto load = [&](int base) {
#pragma unroll
    for (int i = 0; i < RS_BATCH; ++i) {
      const int row = base + i * n_rows;
      s[i] = start > 0 && active && row < p.np ? __ldcs(st + (long long)row * quads) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(row0);  // on its way during the rotation
  const float* ur = u + (long long)b * p.ld;
  const int half = p.rot_dims / 2;
  for (int i = tid; i < 2 * p.np; i += RS_THREADS) {
    const bool key = i >= p.np;
    const int c = key ? i - p.np : i;
    const float* x = ur + ((key ? p.heads : 0) + h) * p.np;
    float v = x[c];
    if (c < p.rot_dims) {
      const int k = c < half ? c : c - half;
      float sn, cs;
      sincosf((float)start * p.freq[k], &sn, &cs);
      v = c < half ? v * cs - x[c + half] * sn : v * cs + x[k] * sn;
    }
    rs_sm[i] = key ? v * p.key_scale : v;
  }
  const float* vr = ur + 2 * p.heads * p.np + h * p.vdp;
  const float* gr = vr + p.heads * p.vdp;
  for (int i = tid; i < p.vdp; i += RS_THREADS) sv[i] = vr[i];
  const float a = p.decay[h];
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    const float4 x = *reinterpret_cast<const float4*>(sv + 4 * quad);
    for (int base = row0;;) {
#pragma unroll
      for (int i = 0; i < RS_BATCH; ++i) {
        const int row = base + i * n_rows;
        if (row >= p.np) break;
        const float kn = sk[row], qn = sq[row];
        float4 v = s[i];
        v.x = fmaf(a, v.x, x.x * kn);
        v.y = fmaf(a, v.y, x.y * kn);
        v.z = fmaf(a, v.z, x.z * kn);
        v.w = fmaf(a, v.w, x.w * kn);
        __stcs(st + (long long)row * quads, v);
        acc.x = fmaf(v.x, qn, acc.x);
        acc.y = fmaf(v.y, qn, acc.y);
        acc.z = fmaf(v.z, qn, acc.z);
        acc.w = fmaf(v.w, qn, acc.w);
      }
      base += RS_BATCH * n_rows;
      if (base >= p.np) break;
      load(base);
    }
    *reinterpret_cast<float4*>(part + 4 * (row0 * quads + quad)) = acc;
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = tid; i < p.vdp; i += RS_THREADS) {
    float v = 0.f;
    for (int r = 0; r < n_rows; ++r) v += part[r * p.vdp + i];
    sv[i] = v;
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < RS_THREADS / 32; ++i) ss += red[i];
  const float f = 1.f / sqrtf(ss / (float)p.vdim + p.eps);
  for (int i = tid; i < p.vdp; i += RS_THREADS) yr[i] = from_f32<T>(sv[i] * f * ss_silu(gr[i]));
}

}  // namespace kvb

#define KVB_RETENTION_TYPES(dtype, ...)                       \
  switch (dtype) {                                            \
    case 0: { using T = float; __VA_ARGS__; break; }          \
    case 1: { using T = __nv_bfloat16; __VA_ARGS__; break; }  \
    default: return KVB_ERR_ARG;                              \
  }

extern "C" int kvb_retention_prep(const float* in, long long ld, const float* freq, void* out, const int* start, int B, int T_, int heads,
                                  int np, int rot_dims, float key_scale, int dtype, void* stream) {
  if (B <= 0 || B > 65535 || T_ <= 0 || heads <= 0 || np <= 0 || ld < 2LL * heads * np || rot_dims < 0 || rot_dims > np || rot_dims % 2)
    return KVB_ERR_ARG;
  if (np % 8 || ld % 4 || (reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out)) & 15) return KVB_ERR_ALIGN;
  kvb::RetPrepParams p;
  p.freq = freq; p.start = start; p.ld = ld; p.T = T_; p.heads = heads; p.np = np; p.rot_dims = rot_dims; p.key_scale = key_scale;
  const size_t smem = (size_t)rot_dims * sizeof(float) + 8;
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  const dim3 grid(T_, B);
  cudaStream_t s = (cudaStream_t)stream;
  KVB_RETENTION_TYPES(dtype, if (rot_dims % 8 == 0) kvb::retention_prep_kernel<T, 4><<<grid, kvb::RP_THREADS, smem, s>>>(in, (T*)out, p);
                      else kvb::retention_prep_kernel<T, 1><<<grid, kvb::RP_THREADS, smem, s>>>(in, (T*)out, p));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_head_norm_gate(const void* y, const void* gate, long long ld, const float* weight, void* out, long long n, int heads, int vdim, int vdp,
                                  float eps, int dtype, void* stream) {
  if (n <= 0 || heads <= 0 || vdim <= 0 || vdp < vdim || n * heads > 0x7f000000LL) return KVB_ERR_ARG;
  if (vdp % 8 || ld % 8 || (reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) & 15)
    return KVB_ERR_ALIGN;
  kvb::HeadNormParams p;
  p.weight = weight; p.ld = ld; p.rows = n * heads; p.heads = heads; p.vdim = vdim; p.vdp = vdp; p.eps = eps;
  KVB_RETENTION_TYPES(dtype, return kvb::hn_type<T>(y, gate, out, p, (cudaStream_t)stream));
}

extern "C" int kvb_retention_step(const float* u, long long ld, const float* freq, const float* decay, float* state, void* out,
                                  const int* slots, const int* start, const int* count, int B, int heads, int vdim, int vdp, int np,
                                  int rot_dims, float key_scale, float eps, int dtype, void* stream) {
  if (B <= 0 || B > 65535 || heads <= 0 || vdim <= 0 || vdp < vdim || np <= 0 || ld < 2LL * heads * (np + vdp) || rot_dims < 0 || rot_dims > np ||
      rot_dims % 2)
    return KVB_ERR_ARG;
  if (vdp % 8 || np % 8) return KVB_ERR_ALIGN;
  if (vdp > 4 * kvb::RS_THREADS) return KVB_ERR_TOO_LARGE;
  const size_t smem = ((size_t)vdp + 2 * np + 4 * kvb::RS_THREADS) * sizeof(float);
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  kvb::RetStepParams p;
  p.freq = freq; p.decay = decay; p.slots = slots; p.start = start; p.count = count; p.state = state; p.ld = ld; p.heads = heads;
  p.vdim = vdim; p.vdp = vdp; p.np = np; p.rot_dims = rot_dims; p.key_scale = key_scale; p.eps = eps;
  KVB_RETENTION_TYPES(dtype, (kvb::retention_step_kernel<T><<<dim3(heads, B), kvb::RS_THREADS, smem, (cudaStream_t)stream>>>(u, (T*)out, p)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
