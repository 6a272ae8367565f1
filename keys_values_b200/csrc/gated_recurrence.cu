// Gated recurrence per channel: S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t x_t with log2 a_t = rate · r_t, gates r and i sigmoids; the result is
// S · gelu(y).
//
//   scan   several new tokens, behind the convolution (ssm.cu) and the gates' products: a cluster of up to eight CTAs has 64 channels of one
//          sequence and takes 64 tokens per CTA at a time. A warp has 8 of them and a lane two channels: decays and additions stay in registers;
//          the warps of a CTA, then the CTAs (asynchronous stores to distributed shared memory) exchange what their tokens make of a state, and
//          every warp runs through its tokens from the right start. Everything is read once;
//   step   one new token per sequence: convolution, gates (a part's products on CUDA cores, weights read once for eight sequences), recurrence
//          and output in one kernel. The inputs of the convolution lie in a ring with one row more than it looks back, so CTAs that share
//          a part do not disturb each other.
//
// Everything from the gates' products on is fp32.
#include <cooperative_groups.h>

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

// The same for results that are rounded to 16 bits, for two channels: few special-function results and paired multiply-adds. Gates in units of
// log2: e = 2^-z, and both sigmoids 1 / (1 + e) come out of one reciprocal; rate2 = 2 ln 2 · rate.
constexpr float GR_LOG2E = 1.4426950408889634f;
__device__ __forceinline__ float gr_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gr_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gr_sqrt(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float2 gr_both(float v) { return make_float2(v, v); }

__device__ __forceinline__ void gr_token2(float2 zr, float2 zi, float2 x, float2 br, float2 bi, float2 rate, float2 rate2, float2& a, float2& add) {
  const float2 ur = ffma2(zr, gr_both(-GR_LOG2E), br), ui = ffma2(zi, gr_both(-GR_LOG2E), bi);
  // 2^60 and beyond: a closed gate either way, and the product stays a number
  const float2 dr = fadd2(make_float2(gr_exp2(fminf(ur.x, 60.f)), gr_exp2(fminf(ur.y, 60.f))), gr_both(1.f));
  const float2 di = fadd2(make_float2(gr_exp2(fminf(ui.x, 60.f)), gr_exp2(fminf(ui.y, 60.f))), gr_both(1.f));
  const float2 d = fmul2(dr, di), inv = make_float2(gr_rcp(d.x), gr_rcp(d.y));
  const float2 r = fmul2(di, inv), i = fmul2(dr, inv);
  const float2 log2a = fmul2(rate, r), w = fmul2(rate2, r);  // w = 2 log a
  a = make_float2(gr_exp2(log2a.x), gr_exp2(log2a.y));
  // 1 - a^2 = 1 - e^w, near zero by the series
  float2 s = ffma2(w, gr_both(1.f / 120.f), gr_both(1.f / 24.f));
  s = ffma2(s, w, gr_both(1.f / 6.f));
  s = ffma2(s, w, gr_both(0.5f));
  s = ffma2(s, w, gr_both(1.f));
  s = fmul2(s, make_float2(-w.x, -w.y));
  const float2 na = make_float2(-a.x, -a.y), far = ffma2(na, a, gr_both(1.f));
  const float2 rest = make_float2(w.x < -0.1f ? far.x : s.x, w.y < -0.1f ? far.y : s.y);
  add = fmul2(fmul2(make_float2(gr_sqrt(rest.x), gr_sqrt(rest.y)), i), x);
}

// z · sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3))
__device__ __forceinline__ float2 gr_gelu2(float2 z) {
  constexpr float K = -1.5957691216057308f * GR_LOG2E;
  const float2 u = fmul2(z, ffma2(fmul2(z, z), gr_both(0.044715f * K), gr_both(K)));
  const float2 d = fadd2(make_float2(gr_exp2(u.x), gr_exp2(u.y)), gr_both(1.f));
  return fmul2(z, make_float2(gr_rcp(d.x), gr_rcp(d.y)));
}

// ------------------------------------------------------------------------------------------------ scan
constexpr int GR_WARPS = 8;
constexpr int GR_RUN = 8;    // tokens of a warp
constexpr int GR_COLS = 64;  // channels of a CTA
constexpr int GR_STEP = GR_WARPS * GR_RUN;
constexpr int GR_CLUSTER = 8;

struct GrScanParams {
  kvb_gated_recurrence g;
  const int *slots, *start, *count;
  const float* z;
  float* state;
  long long ldy, ldo;
  int B, T;
  int* status;
};

template <typename T>
struct alignas(2 * sizeof(T)) GrPair {
  T v[2];
};

// what tokens make of the states of two channels: s -> decay · s + sum
struct alignas(16) GrMade {
  float2 decay, sum;
};
// to the same place of another CTA's shared memory, whose barrier counts the bytes
__device__ __forceinline__ void gr_send(const GrMade* place, uint64_t* bar, int rank, const GrMade& m) {
  uint32_t to, at;
  asm("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(to) : "r"(smem_u32(place)), "r"(rank));
  asm("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(at) : "r"(smem_u32(bar)), "r"(rank));
  asm volatile("st.async.weak.shared::cluster.mbarrier::complete_tx::bytes.v4.b32 [%0], {%1, %2, %3, %4}, [%5];" ::"r"(to),
               "r"(__float_as_uint(m.decay.x)), "r"(__float_as_uint(m.decay.y)), "r"(__float_as_uint(m.sum.x)), "r"(__float_as_uint(m.sum.y)), "r"(at)
               : "memory");
}
__device__ __forceinline__ float2 gr_apply(const GrMade& m, float2 s) { return ffma2(m.decay, s, m.sum); }
__device__ __forceinline__ GrMade gr_then(const GrMade& a, const GrMade& b) { return {fmul2(a.decay, b.decay), ffma2(b.decay, a.sum, b.sum)}; }

template <typename T>
__global__ void __launch_bounds__(GR_WARPS * 32, 2)
gated_recurrence_scan_kernel(const T* __restrict__ x, const T* __restrict__ y, T* __restrict__ out, const GrScanParams p) {
  __shared__ GrMade by_warp[2][GR_WARPS][32], by_cta[2][GR_CLUSTER][32];
  __shared__ uint64_t arrived[2];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  cooperative_groups::cluster_group cluster = cooperative_groups::this_cluster();
  const int rank = (int)cluster.block_rank(), ranks = (int)cluster.num_blocks();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, b = blockIdx.z;
  const int channels = p.g.blocks * p.g.pp, c = blockIdx.y * GR_COLS + 2 * lane;
  const bool mine = c < channels;  // parts are multiples of 8: both channels are of one
  const int cc = mine ? c : 0, part = cc / p.g.pp, j = cc - part * p.g.pp;
  const int n = p.count[b];
  const long long row0 = (long long)b * p.T;
  const float* z = p.z + ((long long)part * p.B * p.T + row0) * 2 * p.g.pp + j;
  x += row0 * channels + cc;
  y += row0 * p.ldy + cc;
  out += row0 * p.ldo + cc;
  constexpr bool HALF = sizeof(T) == 2;
  const float2 rate = *reinterpret_cast<const float2*>(p.g.rate + cc), rate2 = fmul2(rate, gr_both(2.f * GR_LN2));
  float2 br = *reinterpret_cast<const float2*>(p.g.bias_r + cc), bi = *reinterpret_cast<const float2*>(p.g.bias_i + cc);
  if (HALF) {
    br = fmul2(br, gr_both(-GR_LOG2E));
    bi = fmul2(bi, gr_both(-GR_LOG2E));
  }
  const float2 scale = gr_both(p.g.scale);
  float2* own = reinterpret_cast<float2*>(p.state + (long long)p.slots[b] * channels + cc);
  float2 carry = mine && p.start[b] > 0 ? *own : make_float2(0.f, 0.f);
  const GrMade nothing = {make_float2(1.f, 1.f), make_float2(0.f, 0.f)};
  if (ranks > 1) {
    if (threadIdx.x == 0) {
      mbar_init(&arrived[0], 1);
      mbar_init(&arrived[1], 1);
      *abort_flag = 0;
      mbar_fence_init();
    }
    cluster.sync();
  }
  bool ok = true;  // after a wait that ran out the work goes on with what there is: the status word tells
  int turn = 0, phase = 0;
  for (int t0 = 0; t0 < n; t0 += ranks * GR_STEP, turn ^= 1, phase += turn == 0) {
    // Buffers in turn are enough: a CTA that sends for the turn after next has got everybody's results of the next one, which they send after
    // they have read those of this one
    if (ranks > 1 && threadIdx.x == 0) mbar_expect_tx(&arrived[turn], (uint32_t)(ranks * 32 * sizeof(GrMade)));
    const int t1 = t0 + rank * GR_STEP + warp * GR_RUN;
    float2 a[GR_RUN], add[GR_RUN];
    GrPair<T> xv[GR_RUN], yv[GR_RUN];
    const float* zt = z + (long long)t1 * 2 * p.g.pp;
    const T *xt = x + (long long)t1 * channels, *yt = y + (long long)t1 * p.ldy;
    const int have = mine ? min(GR_RUN, n - t1) : 0;  // tokens of this warp
    auto load = [&](int i) {
      a[i] = __ldcs(reinterpret_cast<const float2*>(zt + i * 2 * p.g.pp));
      add[i] = __ldcs(reinterpret_cast<const float2*>(zt + i * 2 * p.g.pp + p.g.pp));
      xv[i] = *reinterpret_cast<const GrPair<T>*>(xt + i * channels);
      yv[i] = *reinterpret_cast<const GrPair<T>*>(yt + i * p.ldy);
    };
    if (have == GR_RUN) {
#pragma unroll
      for (int i = 0; i < GR_RUN; ++i) load(i);
    } else {
#pragma unroll
      for (int i = 0; i < GR_RUN; ++i) {
        a[i] = add[i] = make_float2(0.f, 0.f);
        xv[i].v[0] = xv[i].v[1] = yv[i].v[0] = yv[i].v[1] = from_f32<T>(0.f);
        if (i < have) load(i);
      }
    }
    GrMade own_tokens = nothing;
#pragma unroll
    for (int i = 0; i < GR_RUN; ++i) {
      const float2 xi = make_float2(to_f32(xv[i].v[0]), to_f32(xv[i].v[1]));
      if constexpr (HALF) {
        gr_token2(a[i], add[i], xi, br, bi, rate, rate2, a[i], add[i]);
      } else {
        gr_token<T>(a[i].x + br.x, add[i].x + bi.x, xi.x, rate.x, a[i].x, add[i].x);
        gr_token<T>(a[i].y + br.y, add[i].y + bi.y, xi.y, rate.y, a[i].y, add[i].y);
      }
      if (i >= have) {  // changes nothing
        a[i] = make_float2(1.f, 1.f);
        add[i] = make_float2(0.f, 0.f);
      }
      own_tokens = gr_then(own_tokens, {a[i], add[i]});
    }
    by_warp[turn][warp][lane] = own_tokens;
    __syncthreads();
    GrMade before = nothing, all = nothing;
#pragma unroll
    for (int w = 0; w < GR_WARPS; ++w) {
      if (w == warp) before = all;
      all = gr_then(all, by_warp[turn][w][lane]);
    }
    if (ranks > 1) {  // every CTA of the cluster gets what the others' tokens make of a state
      if (warp < ranks) gr_send(&by_cta[turn][rank][lane], &arrived[turn], warp, all);
      if (ok) ok = mbar_wait_bounded(&arrived[turn], (uint32_t)(phase & 1), abort_flag, p.status, STATUS_TIMEOUT_FULL);
      float2 s = carry;
      for (int r = 0; r < ranks; ++r) {
        if (r == rank) s = carry;
        carry = gr_apply(by_cta[turn][r][lane], carry);
      }
      before = {before.decay, gr_apply(before, s)};
    } else {
      before.sum = gr_apply(before, carry);
      carry = gr_apply(all, carry);
    }
    float2 s = before.sum;
    T* ot = out + (long long)t1 * p.ldo;
#pragma unroll
    for (int i = 0; i < GR_RUN; ++i) {
      s = ffma2(a[i], s, add[i]);
      const float2 yi = make_float2(to_f32(yv[i].v[0]), to_f32(yv[i].v[1]));
      const float2 g = HALF ? gr_gelu2(yi) : make_float2(gr_gelu<T>(yi.x), gr_gelu<T>(yi.y));
      const float2 v = fmul2(fmul2(s, g), scale);
      GrPair<T> o;
      o.v[0] = from_f32<T>(v.x);
      o.v[1] = from_f32<T>(v.y);
      if (i < have) *reinterpret_cast<GrPair<T>*>(ot + i * p.ldo) = o;
    }
  }
  if (ranks > 1) cluster.sync();  // nobody writes into the memory of a CTA that has gone
  if (!mine) return;
  GrPair<T> zero;
  zero.v[0] = zero.v[1] = from_f32<T>(0.f);
  for (int t = n + rank * GR_WARPS + warp; t < p.T; t += ranks * GR_WARPS) *reinterpret_cast<GrPair<T>*>(out + (long long)t * p.ldo) = zero;
  if (rank == 0 && warp == 0 && n > 0) *own = carry;
}

template <typename T>
static int gr_scan_launch(const void* x, const void* y, void* out, const GrScanParams& p, cudaStream_t s) {
  const int tiles = (p.g.blocks * p.g.pp + GR_COLS - 1) / GR_COLS, steps = (p.T + GR_STEP - 1) / GR_STEP;
  int ranks = 1;
  while (ranks < GR_CLUSTER && ranks < steps) ranks *= 2;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(ranks, tiles, p.B);
  cfg.blockDim = dim3(GR_WARPS * 32);
  cfg.stream = s;
  cudaLaunchAttribute attr;
  attr.id = cudaLaunchAttributeClusterDimension;
  attr.val.clusterDim.x = ranks;
  attr.val.clusterDim.y = attr.val.clusterDim.z = 1;
  cfg.attrs = &attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, gated_recurrence_scan_kernel<T>, (const T*)x, (const T*)y, (T*)out, p) == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

// ------------------------------------------------------------------------------------------------ step
constexpr int GQ_ROWS = 8;    // sequences of a CTA, one per warp for the convolution
constexpr int GQ_COLS = 32;   // channels of a CTA, all of one part
constexpr int GQ_SPLIT = 8;   // threads that share a product of two neighbouring channels
constexpr int GQ_THREADS = GQ_COLS * GQ_SPLIT;
constexpr int GQ_TAPS = 4;    // taps of the convolution without a loop
constexpr int GQ_CHANNELS = 4;
constexpr int GQ_AHEAD = 16;  // weights of a thread that are on their way during the convolution

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
  const int pp = p.g.pp, channels = p.g.blocks * pp, taps = p.g.taps, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rows = min(GQ_ROWS, p.B - b0);
  // thread (pair, split): two neighbouring columns of the decay gates (pairs below 16) or input gates, every GQ_SPLIT-th input
  const int pair = tid % GQ_COLS, split = tid / GQ_COLS, col = 2 * (pair % (GQ_COLS / 2)), j = j0 + col;
  const T* w = static_cast<const T*>(p.g.gates) + (long long)part * pp * 2 * pp + (pair < GQ_COLS / 2 ? 0 : pp) + j;
  GrPair<T> ahead[GQ_AHEAD];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int i = 0; i < GQ_AHEAD; ++i) {
      const int k = k0 + i * GQ_SPLIT;
      if (j < pp && k < pp) ahead[i] = *reinterpret_cast<const GrPair<T>*>(w + (long long)k * 2 * pp);
      else ahead[i].v[0] = ahead[i].v[1] = from_f32<T>(0.f);
    }
  };
  fetch(split);
  {
    const bool in = warp < rows;
    const int b = b0 + (in ? warp : 0), pos = p.start[b];
    const bool write = in && p.count[b] > 0;
    T* past = ring + (long long)p.slots[b] * taps * channels + part * pp;
    const T* now = u + b * p.ld + channels + part * pp;
    const float* cw = p.g.conv + part * pp;
    // rows of the ring by how far back they are; up to GQ_TAPS of them, and a run of channels, are on their way together
    int row[GQ_TAPS];
#pragma unroll
    for (int q = 1; q < GQ_TAPS; ++q) row[q] = q < taps && q <= pos ? (pos - q) % taps * channels : -1;
    for (int k0 = lane; k0 < pp; k0 += 32 * GQ_CHANNELS) {
      T x[GQ_CHANNELS], v[GQ_CHANNELS][GQ_TAPS];
      float w[GQ_CHANNELS][GQ_TAPS], bias[GQ_CHANNELS];
#pragma unroll
      for (int i = 0; i < GQ_CHANNELS; ++i) {
        const int k = k0 + 32 * i;
        const bool there = in && k < pp;
        x[i] = from_f32<T>(0.f);
        bias[i] = w[i][0] = 0.f;
        if (there) {
          x[i] = now[k];
          bias[i] = p.g.conv_bias[part * pp + k];
          w[i][0] = cw[(long long)(taps - 1) * channels + k];
        }
#pragma unroll
        for (int q = 1; q < GQ_TAPS; ++q) {
          v[i][q] = from_f32<T>(0.f);
          w[i][q] = 0.f;
          if (there && row[q] >= 0) {
            v[i][q] = past[row[q] + k];
            w[i][q] = cw[(long long)(taps - 1 - q) * channels + k];
          }
        }
      }
#pragma unroll
      for (int i = 0; i < GQ_CHANNELS; ++i) {
        const int k = k0 + 32 * i;
        if (k >= pp) break;
        float s = fmaf(w[i][0], to_f32(x[i]), bias[i]);
#pragma unroll
        for (int q = 1; q < GQ_TAPS; ++q) s = fmaf(w[i][q], to_f32(v[i][q]), s);
        for (int q = GQ_TAPS; in && q < taps && q <= pos; ++q)
          s = fmaf(cw[(long long)(taps - 1 - q) * channels + k], to_f32(past[(long long)((pos - q) % taps) * channels + k]), s);
        // rounded as the product of several tokens reads it
        gq_x[k * GQ_ROWS + warp] = in ? to_f32(from_f32<T>(s)) : 0.f;
        if (write && k >= j0 && k < j0 + GQ_COLS) past[(long long)(pos % taps) * channels + k] = x[i];
      }
    }
  }
  __syncthreads();
  {
    float2 acc[GQ_ROWS];
#pragma unroll
    for (int r = 0; r < GQ_ROWS; ++r) acc[r] = make_float2(0.f, 0.f);
    for (int k0 = split; k0 < pp;) {
#pragma unroll
      for (int i = 0; i < GQ_AHEAD; ++i) {
        const int k = k0 + i * GQ_SPLIT;
        if (k >= pp) break;
        const float2 f = make_float2(to_f32(ahead[i].v[0]), to_f32(ahead[i].v[1]));
        const float4 lo = *reinterpret_cast<const float4*>(gq_x + k * GQ_ROWS), hi = *reinterpret_cast<const float4*>(gq_x + k * GQ_ROWS + 4);
        const float v[GQ_ROWS] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
#pragma unroll
        for (int r = 0; r < GQ_ROWS; ++r) acc[r] = ffma2(f, make_float2(v[r], v[r]), acc[r]);
      }
      k0 += GQ_AHEAD * GQ_SPLIT;
      if (k0 < pp) fetch(k0);
    }
#pragma unroll
    for (int r = 0; r < GQ_ROWS; ++r) *reinterpret_cast<float2*>(&zs[split][r][(pair < GQ_COLS / 2 ? 0 : GQ_COLS) + col]) = acc[r];
  }
  __syncthreads();
  const int jj = j0 + lane, c = part * pp + jj;  // a warp finishes a sequence
  if (warp >= rows || jj >= pp) return;
  const int b = b0 + warp;
  T* dst = out + b * p.ldo + c;
  if (p.count[b] <= 0) {
    *dst = from_f32<T>(0.f);
    return;
  }
  float zr = p.g.bias_r[c], zi = p.g.bias_i[c], a, add;
#pragma unroll
  for (int s = 0; s < GQ_SPLIT; ++s) {
    zr += zs[s][warp][lane];
    zi += zs[s][warp][GQ_COLS + lane];
  }
  gr_token<float>(zr, zi, gq_x[jj * GQ_ROWS + warp], p.g.rate[c], a, add);
  float* own = p.state + (long long)p.slots[b] * channels + c;
  const float s = fmaf(a, p.start[b] > 0 ? *own : 0.f, add);
  *own = s;
  *dst = from_f32<T>(s * gr_gelu<float>(to_f32(u[b * p.ld + c])) * p.g.scale);
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
                                         void* out, long long ldo, const int* slots, const int* start, const int* count, int B, int T_, int dtype, int* status,
                                         void* stream) {
  if (!kvb::gated_recurrence_valid(g) || !z || B <= 0 || B > 65535 || T_ <= 0 || ldy < (long long)g->blocks * g->pp || ldo < (long long)g->blocks * g->pp)
    return KVB_ERR_ARG;
  kvb::GrScanParams p;
  p.g = *g; p.slots = slots; p.start = start; p.count = count; p.z = z; p.state = state; p.ldy = ldy; p.ldo = ldo; p.B = B; p.T = T_; p.status = status;
  if (g->pp % 8 || ldy % 2 || ldo % 2 || (reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(y) |
                                          reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(state)) & 7)
    return KVB_ERR_ALIGN;
  KVB_RECURRENCE_TYPES(dtype, return kvb::gr_scan_launch<T>(x, y, out, p, (cudaStream_t)stream));
}

extern "C" int kvb_gated_recurrence_step(const kvb_gated_recurrence* g, const void* u, long long ld, void* ring, float* state, void* out,
                                         long long ldo, const int* slots, const int* start, const int* count, int B, int dtype, void* stream) {
  using namespace kvb;
  if (!gated_recurrence_valid(g) || !g->gates || B <= 0 || ld < 2LL * g->blocks * g->pp || ldo < (long long)g->blocks * g->pp) return KVB_ERR_ARG;
  const size_t smem = (size_t)g->pp * GQ_ROWS * sizeof(float);
  if (smem > 200 * 1024 || B > 65535 * GQ_ROWS) return KVB_ERR_TOO_LARGE;
  if (g->pp % 8 || (reinterpret_cast<uintptr_t>(g->gates) & 7)) return KVB_ERR_ALIGN;
  GrStepParams p;
  p.g = *g; p.slots = slots; p.start = start; p.count = count; p.state = state; p.ld = ld; p.ldo = ldo; p.B = B;
  p.tiles = (g->pp + GQ_COLS - 1) / GQ_COLS;
  const dim3 grid(g->blocks * p.tiles, (B + GQ_ROWS - 1) / GQ_ROWS);
  KVB_RECURRENCE_TYPES(dtype, static PerDeviceOnce once;
                       if (once.first()) cudaFuncSetAttribute(gated_recurrence_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
                       (gated_recurrence_step_kernel<T><<<grid, GQ_THREADS, smem, (cudaStream_t)stream>>>((const T*)u, (T*)ring, (T*)out, p)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
