// Gated recurrence per channel: S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t x_t with log2 a_t = rate · r_t, gates r and i sigmoids; the result is
// S · gelu(y).
//
//   scan   several new tokens, behind the convolution (ssm.cu) and the gates' products: a CTA has 32 channels of one sequence and takes 128 tokens
//          at a time. A warp has 16 of them and a lane one channel: decays and additions stay in registers, the warps exchange what their
//          tokens make of a state, and then every warp runs through its tokens from the right start. Everything is read once;
//   step   one new token per sequence: convolution, gates (a part's products on CUDA cores, weights read once for eight sequences), recurrence
//          and output in one kernel. The inputs of the convolution lie in a ring with one row more than it looks back, so CTAs that share
//          a part do not disturb each other.
//
// Everything from the gates' products on is fp32.
#include "common.cuh"
#include "kvb200_layers.h"
#include "ssm.cuh"

namespace kvb {

template <typename T>
__device__ __forceinline__ float gr_sigmoid(float x) {
  return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-x)) : 1.f / (1.f + expf(-x));
}

// 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))) = z · sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3))
template <typename T>
__device__ __forceinline__ float gr_gelu(float z) {
  return z * gr_sigmoid<T>(1.5957691216057308f * fmaf(0.044715f * z * z, z, z));
}

// -(e^x - 1) for x <= 0: near zero by the series, which keeps its relative precision
__device__ __forceinline__ float gr_one_minus_exp(float x) {
  if (x < -0.25f) return 1.f - __expf(x);
  float s = fmaf(x, 1.f / 5040.f, 1.f / 720.f);
  s = fmaf(s, x, 1.f / 120.f);
  s = fmaf(s, x, 1.f / 24.f);
  s = fmaf(s, x, 1.f / 6.f);
  s = fmaf(s, x, 0.5f);
  s = fmaf(s, x, 1.f);
  return -x * s;
}

constexpr float GR_LN2 = 0.6931471805599453f;

// decay and addition of a token from the raw gates
template <typename T>
__device__ __forceinline__ void gr_token(float zr, float zi, float x, float rate, float& a, float& add) {
  const float log2a = rate * gr_sigmoid<T>(zr);
  float rest;  // 1 - a^2
  if (sizeof(T) == 2) {
    rest = gr_one_minus_exp(2.f * GR_LN2 * log2a);
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(a) : "f"(log2a));
  } else {
    rest = -expm1f(2.f * GR_LN2 * log2a);
    a = exp2f(log2a);
  }
  add = sqrtf(rest) * gr_sigmoid<T>(zi) * x;
}

// ------------------------------------------------------------------------------------------------ scan
constexpr int GR_WARPS = 8;
constexpr int GR_RUN = 16;  // tokens of a warp
constexpr int GR_STEP = GR_WARPS * GR_RUN;

struct GrScanParams {
  kvb_gated_recurrence g;
  const int *slots, *start, *count;
  const float* z;
  float* state;
  long long ldy, ldo;
  int B, T;
};

template <typename T>
__global__ void __launch_bounds__(GR_WARPS * 32)
gated_recurrence_scan_kernel(const T* __restrict__ x, const T* __restrict__ y, T* __restrict__ out, const GrScanParams p) {
  __shared__ float2 made[2][GR_WARPS][32];  // decay and addition of a warp's tokens
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, b = blockIdx.y;
  const int channels = p.g.blocks * p.g.pp, c = blockIdx.x * 32 + lane;
  const bool mine = c < channels;
  const int cc = mine ? c : 0, part = cc / p.g.pp, j = cc - part * p.g.pp;
  const int n = p.count[b];
  const long long row0 = (long long)b * p.T;
  const float* z = p.z + ((long long)part * p.B * p.T + row0) * 2 * p.g.pp + j;
  x += row0 * channels + cc;
  y += row0 * p.ldy + cc;
  out += row0 * p.ldo + cc;
  const float rate = p.g.rate[cc], br = p.g.bias_r[cc], bi = p.g.bias_i[cc];
  float* own = p.state + (long long)p.slots[b] * channels + cc;
  float carry = mine && p.start[b] > 0 ? *own : 0.f;
  int turn = 0;
  for (int t0 = 0; t0 < n; t0 += GR_STEP, turn ^= 1) {
    const int t1 = t0 + warp * GR_RUN;
    float a[GR_RUN], add[GR_RUN];
    T xv[GR_RUN], yv[GR_RUN];
#pragma unroll
    for (int i = 0; i < GR_RUN; ++i) {
      const int t = t1 + i;
      a[i] = add[i] = 0.f;
      xv[i] = yv[i] = from_f32<T>(0.f);
      if (mine && t < n) {
        a[i] = __ldcs(z + (long long)t * 2 * p.g.pp);
        add[i] = __ldcs(z + (long long)t * 2 * p.g.pp + p.g.pp);
        xv[i] = x[(long long)t * channels];
        yv[i] = y[(long long)t * p.ldy];
      }
    }
    float decay = 1.f, sum = 0.f;
#pragma unroll
    for (int i = 0; i < GR_RUN; ++i) {
      if (t1 + i < n) {
        gr_token<T>(a[i] + br, add[i] + bi, to_f32(xv[i]), rate, a[i], add[i]);
      } else {  // changes nothing
        a[i] = 1.f;
        add[i] = 0.f;
      }
      decay *= a[i];
      sum = fmaf(a[i], sum, add[i]);
    }
    made[turn][warp][lane] = make_float2(decay, sum);
    __syncthreads();
    float s = carry;
#pragma unroll
    for (int w = 0; w < GR_WARPS; ++w) {
      const float2 m = made[turn][w][lane];
      if (w == warp) s = carry;
      carry = fmaf(m.x, carry, m.y);
    }
#pragma unroll
    for (int i = 0; i < GR_RUN; ++i) {
      s = fmaf(a[i], s, add[i]);
      if (mine && t1 + i < n) out[(long long)(t1 + i) * p.ldo] = from_f32<T>(s * gr_gelu<T>(to_f32(yv[i])) * p.g.scale);
    }
  }
  if (!mine) return;
  for (int t = n + warp; t < p.T; t += GR_WARPS) out[(long long)t * p.ldo] = from_f32<T>(0.f);
  if (warp == 0 && n > 0) *own = carry;
}

// ------------------------------------------------------------------------------------------------ step
constexpr int GQ_ROWS = 8;    // sequences of a CTA
constexpr int GQ_COLS = 32;   // channels of a CTA, all of one part
constexpr int GQ_SPLIT = 4;   // threads that share a product
constexpr int GQ_THREADS = 2 * GQ_COLS * GQ_SPLIT;

struct GrStepParams {
  kvb_gated_recurrence g;
  const int *slots, *start, *count;
  float* state;
  long long ld, ldo;
  int B, tiles;  // tiles of GQ_COLS channels in a part
};

template <typename T>
__global__ void __launch_bounds__(GQ_THREADS)
gated_recurrence_step_kernel(const T* __restrict__ u, T* __restrict__ ring, T* __restrict__ out, const GrStepParams p) {
  extern __shared__ float gq_x[];  // (pp, GQ_ROWS): inputs behind the convolution
  __shared__ float zs[GQ_SPLIT][GQ_ROWS][2 * GQ_COLS];
  const int part = blockIdx.x / p.tiles, j0 = (blockIdx.x - part * p.tiles) * GQ_COLS, b0 = blockIdx.y * GQ_ROWS;
  const int pp = p.g.pp, channels = p.g.blocks * pp, taps = p.g.taps, tid = threadIdx.x;
  const int rows = min(GQ_ROWS, p.B - b0);
  for (int i = tid; i < pp * GQ_ROWS; i += GQ_THREADS) {
    const int r = i / pp, k = i - r * pp, c = part * pp + k;
    float v = 0.f;
    if (r < rows) {
      const int b = b0 + r, pos = p.start[b];
      T* past = ring + (long long)p.slots[b] * taps * channels + c;
      const T now = u[b * p.ld + channels + c];
      v = fmaf(p.g.conv[(long long)(taps - 1) * channels + c], to_f32(now), p.g.conv_bias[c]);
      for (int q = 1; q < taps; ++q)
        if (pos - q >= 0) v = fmaf(p.g.conv[(long long)(taps - 1 - q) * channels + c], to_f32(past[(long long)((pos - q) % taps) * channels]), v);
      v = to_f32(from_f32<T>(v));  // as the product of several tokens reads it
      if (k >= j0 && k < j0 + GQ_COLS && p.count[b] > 0) past[(long long)(pos % taps) * channels] = now;
    }
    gq_x[k * GQ_ROWS + r] = v;
  }
  __syncthreads();
  {
    const int col = tid % (2 * GQ_COLS), split = tid / (2 * GQ_COLS);
    const int j = j0 + col % GQ_COLS;
    float acc[GQ_ROWS];
#pragma unroll
    for (int r = 0; r < GQ_ROWS; ++r) acc[r] = 0.f;
    if (j < pp) {
      const T* w = static_cast<const T*>(p.g.gates) + (long long)part * pp * 2 * pp + (col < GQ_COLS ? 0 : pp) + j;
#pragma unroll 8
      for (int k = split; k < pp; k += GQ_SPLIT) {
        const float f = to_f32(w[(long long)k * 2 * pp]);
        const float4 lo = *reinterpret_cast<const float4*>(gq_x + k * GQ_ROWS), hi = *reinterpret_cast<const float4*>(gq_x + k * GQ_ROWS + 4);
        acc[0] = fmaf(f, lo.x, acc[0]);
        acc[1] = fmaf(f, lo.y, acc[1]);
        acc[2] = fmaf(f, lo.z, acc[2]);
        acc[3] = fmaf(f, lo.w, acc[3]);
        acc[4] = fmaf(f, hi.x, acc[4]);
        acc[5] = fmaf(f, hi.y, acc[5]);
        acc[6] = fmaf(f, hi.z, acc[6]);
        acc[7] = fmaf(f, hi.w, acc[7]);
      }
    }
#pragma unroll
    for (int r = 0; r < GQ_ROWS; ++r) zs[split][r][col] = acc[r];
  }
  __syncthreads();
  for (int i = tid; i < GQ_ROWS * GQ_COLS; i += GQ_THREADS) {
    const int r = i / GQ_COLS, j = j0 + i % GQ_COLS, c = part * pp + j;
    if (r >= rows || j >= pp) continue;
    const int b = b0 + r;
    T* dst = out + b * p.ldo + c;
    if (p.count[b] <= 0) {
      *dst = from_f32<T>(0.f);
      continue;
    }
    float zr = p.g.bias_r[c], zi = p.g.bias_i[c], a, add;
#pragma unroll
    for (int s = 0; s < GQ_SPLIT; ++s) {
      zr += zs[s][r][i % GQ_COLS];
      zi += zs[s][r][GQ_COLS + i % GQ_COLS];
    }
    gr_token<float>(zr, zi, gq_x[j * GQ_ROWS + r], p.g.rate[c], a, add);
    float* own = p.state + (long long)p.slots[b] * channels + c;
    const float s = fmaf(a, p.start[b] > 0 ? *own : 0.f, add);
    *own = s;
    *dst = from_f32<T>(s * gr_gelu<float>(to_f32(u[b * p.ld + c])) * p.g.scale);
  }
}

static bool gated_recurrence_valid(const kvb_gated_recurrence* g) {
  return g && g->conv && g->conv_bias && g->bias_r && g->bias_i && g->rate && g->blocks > 0 && g->pp > 0 && g->taps > 0;
}

}  // namespace kvb

#define KVB_RECURRENCE_TYPES(dtype, ...)                      \
  switch (dtype) {                                            \
    case 0: { using T = float; __VA_ARGS__; break; }          \
    case 1: { using T = __nv_bfloat16; __VA_ARGS__; break; }  \
    default: return KVB_ERR_ARG;                              \
  }

extern "C" int kvb_gated_recurrence_scan(const kvb_gated_recurrence* g, const void* x, const float* z, const void* y, long long ldy, float* state,
                                         void* out, long long ldo, const int* slots, const int* start, const int* count, int B, int T_, int dtype,
                                         void* stream) {
  if (!kvb::gated_recurrence_valid(g) || !z || B <= 0 || B > 65535 || T_ <= 0 || ldy < (long long)g->blocks * g->pp || ldo < (long long)g->blocks * g->pp)
    return KVB_ERR_ARG;
  kvb::GrScanParams p;
  p.g = *g; p.slots = slots; p.start = start; p.count = count; p.z = z; p.state = state; p.ldy = ldy; p.ldo = ldo; p.B = B; p.T = T_;
  const dim3 grid((g->blocks * g->pp + 31) / 32, B);
  KVB_RECURRENCE_TYPES(dtype, (kvb::gated_recurrence_scan_kernel<T><<<grid, kvb::GR_WARPS * 32, 0, (cudaStream_t)stream>>>(
      (const T*)x, (const T*)y, (T*)out, p)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_gated_recurrence_step(const kvb_gated_recurrence* g, const void* u, long long ld, void* ring, float* state, void* out,
                                         long long ldo, const int* slots, const int* start, const int* count, int B, int dtype, void* stream) {
  using namespace kvb;
  if (!gated_recurrence_valid(g) || !g->gates || B <= 0 || ld < 2LL * g->blocks * g->pp || ldo < (long long)g->blocks * g->pp) return KVB_ERR_ARG;
  const size_t smem = (size_t)g->pp * GQ_ROWS * sizeof(float);
  if (smem > 200 * 1024 || B > 65535 * GQ_ROWS) return KVB_ERR_TOO_LARGE;
  GrStepParams p;
  p.g = *g; p.slots = slots; p.start = start; p.count = count; p.state = state; p.ld = ld; p.ldo = ldo; p.B = B;
  p.tiles = (g->pp + GQ_COLS - 1) / GQ_COLS;
  const dim3 grid(g->blocks * p.tiles, (B + GQ_ROWS - 1) / GQ_ROWS);
  KVB_RECURRENCE_TYPES(dtype, static PerDeviceOnce once;
                       if (once.first()) cudaFuncSetAttribute(gated_recurrence_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
                       (gated_recurrence_step_kernel<T><<<grid, GQ_THREADS, smem, (cudaStream_t)stream>>>((const T*)u, (T*)ring, (T*)out, p)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
