// Gated linear attention: S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t with a decay per token and key channel, alpha =
// sigmoid(z)^(1 / tau), z a low-rank projection with a bias; o normed per head with a weight and gated (norm: retention.cu). The recurrence
// over several tokens is the one of state-space mixers (ssm.cu, ssm_sm100.cu); here are
//
//   prep   chunks of 128 tokens: second half of z's projection, logarithms of the decays and their running sums c_t in fp32. With r the sum up to
//          the middle of the chunk, queries become q exp(c_t - r) and keys k exp(r - c_t), rounded once: within the chunk q_t · k_s then holds the
//          decay from s to t, and the state in units of exp(r) meets both. The factors of a chunk's halves go to the scan. Where a half decays by
//          more than 2^-60 the head is marked, and the plain scan takes it;
//   step   one new token per sequence: decays, state, output, norm and gate of a head in one kernel, all in fp32, bound by reading and writing the
//          state once.
#include "common.cuh"
#include "kvb200_layers.h"
#include "ssm.cuh"

namespace kvb {

constexpr int GL_T = 128;       // tokens of a chunk
constexpr int GL_COLS = 32;     // key channels of a CTA
constexpr int GL_RUN = 8;       // tokens of a thread
constexpr int GL_GROUPS = GL_T / GL_RUN;
constexpr int GL_THREADS = GL_COLS / 4 * GL_GROUPS;
constexpr float GL_FAR = 60.f;  // log2
constexpr float GL_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float gl_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct GlPrepParams {
  kvb_gated_linear g;
  const int* count;
  float* factor;
  int* far;
  int T, lda;
};

__global__ void __launch_bounds__(GL_THREADS)
gated_linear_prep_kernel(__nv_bfloat16* __restrict__ out, const GlPrepParams p) {
  extern __shared__ float gl_a[];  // (GL_T, lda)
  __shared__ float4 sums[GL_GROUPS][GL_COLS / 4];
  const int chunk = blockIdx.x, b = blockIdx.z, n = p.count[b];
  const int lane = threadIdx.x % (GL_COLS / 4), group = threadIdx.x / (GL_COLS / 4);
  const int keys = p.g.heads * p.g.np, c = blockIdx.y * GL_COLS + 4 * lane;
  const bool mine = c < keys;  // np is a multiple of 8: the four channels are of one head
  const int t0 = chunk * GL_T + group * GL_RUN, rank = p.g.rank;
  const long long row0 = (long long)b * p.T;
  for (int i = threadIdx.x; i < GL_T * rank; i += GL_THREADS) {
    const int t = i / rank, r = i - t * rank;
    gl_a[t * p.lda + r] = chunk * GL_T + t < p.T ? p.g.in[(row0 + chunk * GL_T + t) * p.g.ld + 2 * keys + r] : 0.f;
  }
  __syncthreads();
  float4 z[GL_RUN];
  const float4 bias = mine ? *reinterpret_cast<const float4*>(p.g.bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int t = 0; t < GL_RUN; ++t) z[t] = bias;
  const float* a = gl_a + group * GL_RUN * p.lda;
#pragma unroll 4
  for (int r = 0; r < rank; ++r) {
    const float4 w = mine ? *reinterpret_cast<const float4*>(p.g.w + (long long)r * keys + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int t = 0; t < GL_RUN; ++t) {
      const float v = a[t * p.lda + r];
      z[t].x = fmaf(v, w.x, z[t].x);
      z[t].y = fmaf(v, w.y, z[t].y);
      z[t].z = fmaf(v, w.z, z[t].z);
      z[t].w = fmaf(v, w.w, z[t].w);
    }
  }
  // running sums within the thread's tokens; padding decays nothing
  const float f = -p.g.inv_tau * GL_LOG2E;
  float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int t = 0; t < GL_RUN; ++t) {
    if (t0 + t < n) {
      sum.x = fmaf(f, ss_softplus_fast(-z[t].x), sum.x);
      sum.y = fmaf(f, ss_softplus_fast(-z[t].y), sum.y);
      sum.z = fmaf(f, ss_softplus_fast(-z[t].z), sum.z);
      sum.w = fmaf(f, ss_softplus_fast(-z[t].w), sum.w);
    }
    z[t] = sum;
  }
  sums[group][lane] = sum;
  __syncthreads();
  float4 before = make_float4(0.f, 0.f, 0.f, 0.f), half = before, whole = before;
#pragma unroll
  for (int i = 0; i < GL_GROUPS; ++i) {
    const float4 s = sums[i][lane];
    if (i == group) before = whole;
    whole.x += s.x;
    whole.y += s.y;
    whole.z += s.z;
    whole.w += s.w;
    if (i == GL_GROUPS / 2 - 1) half = whole;
  }
  if (!mine) return;
  if (group == 0) {
    const float4 rest = make_float4(whole.x - half.x, whole.y - half.y, whole.z - half.z, whole.w - half.w);
    float4* dst = reinterpret_cast<float4*>(p.factor + (((long long)b * gridDim.x + chunk) * keys + c) * 2);
    dst[0] = make_float4(half.x, rest.x, half.y, rest.y);
    dst[1] = make_float4(half.z, rest.z, half.w, rest.w);
    const float low = fminf(fminf(fminf(half.x, half.y), fminf(half.z, half.w)), fminf(fminf(rest.x, rest.y), fminf(rest.z, rest.w)));
    if (!(low >= -GL_FAR)) p.far[b * p.g.heads + c / p.g.np] = 1;  // several threads, the same value
  }
  const float4 shift = make_float4(before.x - half.x, before.y - half.y, before.z - half.z, before.w - half.w);
  const float qs = p.g.q_scale;
#pragma unroll
  for (int t = 0; t < GL_RUN; ++t) {
    if (t0 + t >= p.T) break;
    __nv_bfloat16* dst = out + (row0 + t0 + t) * 2 * keys + c;
    uint2 qo = make_uint2(0u, 0u), ko = qo;
    if (t0 + t < n) {
      const float* src = p.g.in + (row0 + t0 + t) * p.g.ld + c;
      const float4 q = *reinterpret_cast<const float4*>(src), k = *reinterpret_cast<const float4*>(src + keys);
      float e[4] = {z[t].x + shift.x, z[t].y + shift.y, z[t].z + shift.z, z[t].w + shift.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) e[i] = fminf(fmaxf(e[i], -GL_FAR), GL_FAR);  // marked heads only
      qo = make_uint2(pack_bf16x2(q.x * qs * gl_exp2(e[0]), q.y * qs * gl_exp2(e[1])), pack_bf16x2(q.z * qs * gl_exp2(e[2]), q.w * qs * gl_exp2(e[3])));
      ko = make_uint2(pack_bf16x2(k.x * gl_exp2(-e[0]), k.y * gl_exp2(-e[1])), pack_bf16x2(k.z * gl_exp2(-e[2]), k.w * gl_exp2(-e[3])));
    }
    *reinterpret_cast<uint2*>(dst) = qo;
    *reinterpret_cast<uint2*>(dst + keys) = ko;
  }
}

// ------------------------------------------------------------------------------------------------ step
constexpr int GS_THREADS = 256;
constexpr int GS_BATCH = 8;  // float4 of the state that a thread has in flight

struct GlStepParams {
  kvb_gated_linear g;
  const float* norm;
  const int *slots, *start, *count;
  float* state;
  int v_col, vdim, vdp;
  float eps;
};

// One head of one sequence. Thread (row, quad) has four value columns of rows row, row + n_rows, ...
template <typename T>
__global__ void __launch_bounds__(GS_THREADS)
gated_linear_step_kernel(T* __restrict__ out, const GlStepParams p) {
  extern __shared__ float gs_sm[];  // q (np) | k (np) | decays (np) | v (vdp) | partial sums (GS_THREADS · 4)
  __shared__ float red[GS_THREADS / 32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, np = p.g.np, keys = p.g.heads * np;
  T* yr = out + ((long long)b * p.g.heads + h) * p.vdp;
  if (p.count[b] <= 0) {
    for (int i = tid; i < p.vdp; i += GS_THREADS) yr[i] = from_f32<T>(0.f);
    return;
  }
  float *sq = gs_sm, *sk = sq + np, *sa = sk + np, *sv = sa + np, *part = sv + p.vdp;
  const int quads = p.vdp / 4, n_rows = GS_THREADS / quads;
  const int row0 = tid / quads, quad = tid - row0 * quads;
  const bool active = row0 < n_rows, fresh = p.start[b] == 0;
  float4* st = reinterpret_cast<float4*>(p.state + ((long long)p.slots[b] * p.g.heads + h) * np * p.vdp) + quad;
  float4 s[GS_BATCH];
  auto load = [&](int base) {
#pragma unroll
    for (int i = 0; i < GS_BATCH; ++i) {
      const int row = base + i * n_rows;
      s[i] = !fresh && active && row < np ? __ldcs(st + (long long)row * quads) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(row0);  // on its way while the decays are made
  const float* ur = p.g.in + (long long)b * p.g.ld;
  for (int i = tid; i < np; i += GS_THREADS) {
    const int c = h * np + i;
    sq[i] = ur[c] * p.g.q_scale;
    sk[i] = ur[keys + c];
    sa[i] = ss_decay(gl_log_decay(p.g, ur + 2 * keys, c));
  }
  const float* vr = ur + p.v_col + h * p.vdp;
  const float* gr = vr + p.g.heads * p.vdp;
  for (int i = tid; i < p.vdp; i += GS_THREADS) sv[i] = vr[i];
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    const float4 x = *reinterpret_cast<const float4*>(sv + 4 * quad);
    for (int base = row0;;) {
#pragma unroll
      for (int i = 0; i < GS_BATCH; ++i) {
        const int row = base + i * n_rows;
        if (row >= np) break;
        const float kn = sk[row], qn = sq[row], a = sa[row];
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
      base += GS_BATCH * n_rows;
      if (base >= np) break;
      load(base);
    }
    *reinterpret_cast<float4*>(part + 4 * (row0 * quads + quad)) = acc;
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = tid; i < p.vdp; i += GS_THREADS) {
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
  for (int i = 0; i < GS_THREADS / 32; ++i) ss += red[i];
  const float f = 1.f / sqrtf(ss / (float)p.vdim + p.eps);
  for (int i = tid; i < p.vdp; i += GS_THREADS) yr[i] = from_f32<T>(sv[i] * f * p.norm[i] * ss_silu(gr[i]));
}

static bool gated_linear_valid(const kvb_gated_linear* g) {
  return g && g->in && g->w && g->bias && g->heads > 0 && g->np > 0 && g->rank > 0 && g->ld >= 2LL * g->heads * g->np + g->rank;
}

}  // namespace kvb

extern "C" int kvb_gated_linear_prep(const kvb_gated_linear* g, void* out, float* factor, int* far, const int* count, int B, int T, void* stream) {
  using namespace kvb;
  if (!gated_linear_valid(g) || B <= 0 || B > 65535 || T <= 0) return KVB_ERR_ARG;
  if (g->np % 8 || g->ld % 4 || (reinterpret_cast<uintptr_t>(g->in) | reinterpret_cast<uintptr_t>(g->w) | reinterpret_cast<uintptr_t>(g->bias) |
                                 reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(factor)) & 15)
    return KVB_ERR_ALIGN;
  GlPrepParams p;
  p.g = *g; p.count = count; p.factor = factor; p.far = far; p.T = T; p.lda = g->rank | 1;
  const size_t smem = (size_t)GL_T * p.lda * sizeof(float);
  const long long keys = (long long)g->heads * g->np;
  if (smem > 200 * 1024 || keys > GL_COLS * 65535LL) return KVB_ERR_TOO_LARGE;
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(gated_linear_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  cudaStream_t s = (cudaStream_t)stream;
  if (cudaMemsetAsync(far, 0, sizeof(int) * B * g->heads, s) != cudaSuccess) return KVB_ERR_CUDA;
  const dim3 grid((T + GL_T - 1) / GL_T, (unsigned)((keys + GL_COLS - 1) / GL_COLS), B);
  gated_linear_prep_kernel<<<grid, GL_THREADS, smem, s>>>((__nv_bfloat16*)out, p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_gated_linear_step(const kvb_gated_linear* g, int v_col, const float* norm, float* state, void* out, const int* slots,
                                     const int* start, const int* count, int B, int vdim, int vdp, float eps, int dtype, void* stream) {
  using namespace kvb;
  if (!gated_linear_valid(g) || B <= 0 || B > 65535 || vdim <= 0 || vdp < vdim || v_col < 2 * g->heads * g->np + g->rank || !norm ||
      g->ld < v_col + 2LL * g->heads * vdp)
    return KVB_ERR_ARG;
  if (vdp % 8 || g->np % 8) return KVB_ERR_ALIGN;
  if (vdp > 4 * GS_THREADS) return KVB_ERR_TOO_LARGE;
  const size_t smem = ((size_t)vdp + 3 * g->np + 4 * GS_THREADS) * sizeof(float);
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  GlStepParams p;
  p.g = *g; p.norm = norm; p.slots = slots; p.start = start; p.count = count; p.state = state; p.v_col = v_col; p.vdim = vdim; p.vdp = vdp;
  p.eps = eps;
  const dim3 grid(g->heads, B);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == 0) gated_linear_step_kernel<float><<<grid, GS_THREADS, smem, s>>>((float*)out, p);
  else if (dtype == 1) gated_linear_step_kernel<__nv_bfloat16><<<grid, GS_THREADS, smem, s>>>((__nv_bfloat16*)out, p);
  else return KVB_ERR_ARG;
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
