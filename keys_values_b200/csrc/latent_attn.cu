// Latent attention: queries of H heads against one latent per token (plus one rotated key part that the heads share).
//
//   prep    splits the joint projection, norms the latent, rotates the rotary parts (angles in fp32, computed once per
//           token), writes padded query and latent rows, the latter to the buffer of the pass and into the ring;
//   ring    a layer that sees a window of W tokens keeps W latents per sequence: position p lives in slot p mod length;
//   attend  several new tokens: keys and values of the window before the pass and of the pass itself are expanded from
//           the latents by a matrix product and swept with an online softmax (here on CUDA cores, for fp32 and for shapes the
//           tcgen05 kernel of latent_sm100.cu does not take);
//   decode  one new token per sequence stays in latent space: W_uk is folded into the query and W_uv into the output, so
//           the ring is read once for all heads and serves as key and value.
#include <cuda.h>

#include "common.cuh"
#include "kvb200_layers.h"
#include "tmap.cuh"

namespace kvb {

// ------------------------------------------------------------------------------------------------ prep
// A CTA has RUN consecutive tokens of a row. First the angles of its tokens and the root mean squares of their latents (one
// warp per token), then the columns that are only copied or normed, then the rotary ones (V elements per access, 16 bytes; 1 when
// the sizes do not divide).
constexpr int LP_THREADS = 256;
constexpr int LP_RUN = 2;  // tokens of a CTA when there are many

template <typename T, int V>
struct alignas(sizeof(T) * V) LpVec {
  T v[V];
};

struct LpParams {
  long long ld;
  const float *norm_w, *freq;
  const int *slots, *start, *count;
  int T, P, ring_len, heads, dim, dimp, rot, rot_dims, rp, kv_rank, kvp;
  unsigned plain_magic, rot_magic;
  float eps;
};

template <typename T, int V, int RUN>
__global__ void __launch_bounds__(LP_THREADS, 6)
latent_prep_kernel(const T* __restrict__ qkv, T* __restrict__ q, T* __restrict__ latent, T* __restrict__ ring, const LpParams p) {
  using Vec = LpVec<T, V>;
  extern __shared__ float sm[];  // per token: cos | sin (rot_dims / 2 each)
  __shared__ float inv_rms[RUN];
  const int t0 = blockIdx.x * RUN, b = blockIdx.y;
  const int nt = min(RUN, p.T - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int start = p.start[b], half = p.rot_dims / 2;
  const int c0 = p.heads * (p.dim + p.rot);
  const long long n0 = (long long)b * p.T + t0;
  for (int i = threadIdx.x; i < nt * half; i += LP_THREADS) {
    const int t = i / half, k = i - t * half;
    sincosf((float)(start + t0 + t) * p.freq[k], &sm[t * p.rot_dims + half + k], &sm[t * p.rot_dims + k]);
  }
  if (warp < nt) {
    const T* c = qkv + (n0 + warp) * p.ld + c0;
    float ss = 0.f;
    for (int i = lane * V; i < p.kv_rank; i += 32 * V) {
      const Vec a = *reinterpret_cast<const Vec*>(c + i);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(to_f32(a.v[e]), to_f32(a.v[e]), ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) inv_rms[warp] = 1.f / sqrtf(ss / (float)p.kv_rank + p.eps);
  }
  __syncthreads();
  const int dq = p.dimp + p.rp, lw = p.kvp + p.rp;
  const int last = p.count[b];
  const T* src0 = qkv + n0 * p.ld;
  // where token t of this CTA has its latent row in the ring: the last ring_len tokens of the pass, no padding
  auto ring_row = [&](int t) -> T* {
    const int tt = t0 + t;
    if (!ring || tt >= last || tt < last - p.ring_len) return nullptr;
    return ring + ((long long)p.slots[b] * p.ring_len + (start + tt) % p.ring_len) * lw;
  };
  auto put_latent = [&](int t, int col, const Vec& v) {
    if (latent) *reinterpret_cast<Vec*>(latent + ((long long)b * (p.P + p.T) + p.P + t0 + t) * lw + col) = v;
    T* r = ring_row(t);
    if (r) *reinterpret_cast<Vec*>(r + col) = v;
  };
  // ---- columns that are not rotated: all tokens are loaded before any is stored
  const int pu = p.dimp / V, pq = p.heads * pu;
  for (int i = threadIdx.x; i < pq; i += LP_THREADS) {
    const int h = pu == 1 ? i : (int)__umulhi((unsigned)i, p.plain_magic), j = (i - h * pu) * V;
    Vec a[RUN];
#pragma unroll
    for (int t = 0; t < RUN; ++t) {
      if (t < nt && j < p.dim) {
        a[t] = *reinterpret_cast<const Vec*>(src0 + t * p.ld + h * (p.dim + p.rot) + j);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) a[t].v[e] = from_f32<T>(0.f);
      }
    }
#pragma unroll
    for (int t = 0; t < RUN; ++t)
      if (t < nt) *reinterpret_cast<Vec*>(q + ((n0 + t) * p.heads + h) * dq + j) = a[t];
  }
  for (int i = threadIdx.x; i < p.kvp / V; i += LP_THREADS) {
    const int j = i * V;
#pragma unroll
    for (int t = 0; t < RUN; ++t) {
      if (t >= nt) break;
      Vec a;
      if (j < p.kv_rank) {
        a = *reinterpret_cast<const Vec*>(src0 + t * p.ld + c0 + j);
        const float r = inv_rms[t];
#pragma unroll
        for (int e = 0; e < V; ++e) a.v[e] = from_f32<T>(to_f32(a.v[e]) * r * p.norm_w[j + e]);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) a.v[e] = from_f32<T>(0.f);
      }
      put_latent(t, j, a);
    }
  }
  // ---- rotary parts of the heads and of the latent row: V pairs per thread, both halves
  const int ru = half / V, rq = (p.heads + 1) * ru;
  for (int i = threadIdx.x; i < rq; i += LP_THREADS) {
    const int h = ru == 1 ? i : (int)__umulhi((unsigned)i, p.rot_magic), k = (i - h * ru) * V;
    const int x = (h < p.heads ? h * (p.dim + p.rot) + p.dim : c0 + p.kv_rank) + k;
#pragma unroll
    for (int t = 0; t < RUN; ++t) {
      if (t >= nt) break;
      Vec a = *reinterpret_cast<const Vec*>(src0 + t * p.ld + x), w = *reinterpret_cast<const Vec*>(src0 + t * p.ld + x + half);
      const float *cs = sm + t * p.rot_dims + k, *sn = cs + half;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float u = to_f32(a.v[e]), v = to_f32(w.v[e]);
        a.v[e] = from_f32<T>(u * cs[e] - v * sn[e]);
        w.v[e] = from_f32<T>(v * cs[e] + u * sn[e]);
      }
      if (h < p.heads) {
        T* d = q + ((n0 + t) * p.heads + h) * dq + p.dimp + k;
        *reinterpret_cast<Vec*>(d) = a;
        *reinterpret_cast<Vec*>(d + half) = w;
      } else {
        put_latent(t, p.kvp + k, a);
        put_latent(t, p.kvp + half + k, w);
      }
    }
  }
  // ---- rotary columns beyond rot_dims pass, padding is zero
  const int tail = p.rp - p.rot_dims;
  for (int i = threadIdx.x; i < (p.heads + 1) * tail * nt; i += LP_THREADS) {
    const int t = i / ((p.heads + 1) * tail), h = i / tail % (p.heads + 1), r = p.rot_dims + i % tail;
    const T v = r < p.rot ? src0[t * p.ld + (h < p.heads ? h * (p.dim + p.rot) + p.dim : c0 + p.kv_rank) + r] : from_f32<T>(0.f);
    if (h < p.heads) {
      q[((n0 + t) * p.heads + h) * dq + p.dimp + r] = v;
    } else {
      if (latent) latent[((long long)b * (p.P + p.T) + p.P + t0 + t) * lw + p.kvp + r] = v;
      T* d = ring_row(t);
      if (d) d[p.kvp + r] = v;
    }
  }
}

template <typename T, int V>
static int lp_launch_run(const void* qkv, void* q, void* latent, void* ring, LpParams& p, int B, cudaStream_t s) {
  // i / n as a high product, exact for i, n < 2^16
  auto magic = [](int n) { return n > 1 ? (unsigned)(0x100000000ull / n + 1) : 0u; };
  p.plain_magic = magic(p.dimp / V);
  p.rot_magic = magic(p.rot_dims / 2 / V);
  if ((long long)p.heads * p.dimp >= 65536 || (long long)(p.heads + 1) * p.rot_dims >= 65536) return KVB_ERR_TOO_LARGE;
  const bool many = (long long)B * p.T >= 148 * 4 * LP_RUN;
  const int run = many ? LP_RUN : 1;
  const size_t smem = (size_t)run * p.rot_dims * sizeof(float) + 8;
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  const dim3 grid((p.T + run - 1) / run, B);
  if (many)
    latent_prep_kernel<T, V, LP_RUN><<<grid, LP_THREADS, smem, s>>>((const T*)qkv, (T*)q, (T*)latent, (T*)ring, p);
  else
    latent_prep_kernel<T, V, 1><<<grid, LP_THREADS, smem, s>>>((const T*)qkv, (T*)q, (T*)latent, (T*)ring, p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

template <typename T>
static int lp_launch(const void* qkv, void* q, void* latent, void* ring, LpParams& p, int B, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  if (((p.dim | p.rot | p.kv_rank | (p.rot_dims / 2)) % V) == 0 && p.ld % V == 0) return lp_launch_run<T, V>(qkv, q, latent, ring, p, B, s);
  return lp_launch_run<T, 1>(qkv, q, latent, ring, p, B, s);
}

// ------------------------------------------------------------------------------------------------ ring
// Rows are multiples of 16 bytes (`units` of them); one warp per row.
constexpr int LR_WARPS = 8;

__global__ void __launch_bounds__(LR_WARPS * 32)
ring_gather_kernel(const uint4* __restrict__ ring, uint4* __restrict__ latent, const int* __restrict__ slots, const int* __restrict__ start,
                   int Tn, int P, int ring_len, int units) {
  const int j = blockIdx.x * LR_WARPS + (threadIdx.x >> 5), b = blockIdx.y;
  if (j >= P) return;
  const int pos = start[b] - P + j;
  uint4* dst = latent + ((long long)b * (P + Tn) + j) * units;
  const bool has = pos >= 0 && pos >= start[b] - ring_len;
  const uint4* src = ring + ((long long)slots[b] * ring_len + (has ? pos % ring_len : 0)) * units;
  for (int i = threadIdx.x & 31; i < units; i += 32) dst[i] = has ? src[i] : make_uint4(0, 0, 0, 0);
}

// ------------------------------------------------------------------- attention over expanded keys, CUDA cores
constexpr int LA_WARPS = 4;
constexpr int LA_MAX_V = 16;  // value features per lane

template <typename T>
__global__ void __launch_bounds__(LA_WARPS * 32)
latent_attend_simple_kernel(const T* __restrict__ q, const T* __restrict__ kv, const T* __restrict__ latent, T* __restrict__ out,
                            const int* __restrict__ start, int Tn, int P, int heads, int dimp, int rp, int kvp, int vdp, int window,
                            float scale) {
  extern __shared__ float qs_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * LA_WARPS + warp, h = blockIdx.y, b = blockIdx.z;
  if (t >= Tn) return;
  const int dq = dimp + rp, lw = kvp + rp, row = dimp + vdp;
  float* qs = qs_all + warp * dq;
  const T* qp = q + (((long long)b * Tn + t) * heads + h) * dq;
  for (int i = lane; i < dq; i += 32) qs[i] = to_f32(qp[i]);
  __syncwarp();
  const int hi = P + t;
  int lo = window > 0 ? hi - window + 1 : 0;
  lo = max(lo, max(0, P - start[b]));
  float m = -INFINITY, l = 0.f;
  float acc[LA_MAX_V];
#pragma unroll
  for (int i = 0; i < LA_MAX_V; ++i) acc[i] = 0.f;
  const long long base = (long long)b * (P + Tn);
  for (int j0 = lo; j0 <= hi; j0 += 32) {
    const int j = j0 + lane;
    float s = -INFINITY;
    if (j <= hi) {
      const T* k = kv + ((base + j) * heads + h) * row;
      const T* kr = latent + (base + j) * lw + kvp;
      float a0 = 0.f, a1 = 0.f;
      for (int i = 0; i < dimp; i += 2) {
        a0 = fmaf(qs[i], to_f32(k[i]), a0);
        a1 = fmaf(qs[i + 1], to_f32(k[i + 1]), a1);
      }
      for (int i = 0; i < rp; i += 2) {
        a0 = fmaf(qs[dimp + i], to_f32(kr[i]), a0);
        a1 = fmaf(qs[dimp + i + 1], to_f32(kr[i + 1]), a1);
      }
      s = (a0 + a1) * scale;
    }
    const float mn = fmaxf(m, warp_max(s));
    const float f = expf(m - mn);
    const float p = expf(s - mn);
    m = mn;
    l = l * f + warp_sum(p);
#pragma unroll
    for (int i = 0; i < LA_MAX_V; ++i) acc[i] *= f;
    const int nk = min(32, hi - j0 + 1);
    for (int e = 0; e < nk; ++e) {
      const float pe = __shfl_sync(0xffffffffu, p, e);
      const T* v = kv + ((base + j0 + e) * heads + h) * row + dimp;
#pragma unroll
      for (int i = 0; i < LA_MAX_V; ++i) {
        const int c = i * 32 + lane;
        if (c < vdp) acc[i] = fmaf(pe, to_f32(v[c]), acc[i]);
      }
    }
  }
  const float inv = 1.f / l;
  T* o = out + (((long long)b * Tn + t) * heads + h) * vdp;
#pragma unroll
  for (int i = 0; i < LA_MAX_V; ++i) {
    const int c = i * 32 + lane;
    if (c < vdp) o[c] = from_f32<T>(acc[i] * inv);
  }
}

// --------------------------------------------------------------------------- single token, CUDA cores
constexpr int LD_MAX_C = 32;  // latent features per lane

template <typename T>
__global__ void __launch_bounds__(128)
latent_decode_simple_kernel(const T* __restrict__ q_abs, const T* __restrict__ q, const T* __restrict__ ring, T* __restrict__ out,
                            const int* __restrict__ slots, const int* __restrict__ start, int B, int heads, int dimp, int rp, int kvp,
                            int ring_len, float scale) {
  extern __shared__ float sm[];  // query (kvp + rp) | partial outputs (4 x kvp) | m, l (4 each)
  const int h = blockIdx.x, b = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int lw = kvp + rp;
  float *qs = sm, *po = qs + lw, *pm = po + 4 * kvp, *pl = pm + 4;
  for (int i = threadIdx.x; i < lw; i += 128)
    qs[i] = i < kvp ? to_f32(q_abs[((long long)h * B + b) * kvp + i])
                    : to_f32(q[((long long)b * heads + h) * (dimp + rp) + dimp + i - kvp]);
  __syncthreads();
  const int nk = min(start[b] + 1, ring_len);
  const T* base = ring + (long long)slots[b] * ring_len * lw;
  float m = -INFINITY, l = 0.f;
  float acc[LD_MAX_C];
#pragma unroll
  for (int i = 0; i < LD_MAX_C; ++i) acc[i] = 0.f;
  for (int j = warp; j < nk; j += 4) {
    const T* k = base + (long long)j * lw;
    float s = 0.f;
    for (int i = lane; i < lw; i += 32) s = fmaf(qs[i], to_f32(k[i]), s);
    s = warp_sum(s) * scale;
    const float mn = fmaxf(m, s);
    const float f = expf(m - mn), p = expf(s - mn);
    m = mn;
    l = l * f + p;
#pragma unroll
    for (int i = 0; i < LD_MAX_C; ++i) {
      const int c = i * 32 + lane;
      if (c < kvp) acc[i] = fmaf(p, to_f32(k[c]), acc[i] * f);
    }
  }
  if (lane == 0) {
    pm[warp] = m;
    pl[warp] = l;
  }
  __syncthreads();
  const float M = fmaxf(fmaxf(pm[0], pm[1]), fmaxf(pm[2], pm[3]));
  const float f = m == -INFINITY ? 0.f : expf(m - M);
#pragma unroll
  for (int i = 0; i < LD_MAX_C; ++i) {
    const int c = i * 32 + lane;
    if (c < kvp) po[warp * kvp + c] = acc[i] * f;
  }
  float L = 0.f;
  for (int w = 0; w < 4; ++w) L += pm[w] == -INFINITY ? 0.f : pl[w] * expf(pm[w] - M);
  __syncthreads();
  for (int c = threadIdx.x; c < kvp; c += 128)
    out[((long long)h * B + b) * kvp + c] = from_f32<T>((po[c] + po[kvp + c] + po[2 * kvp + c] + po[3 * kvp + c]) / L);
}

// ------------------------------------------------------------------ single token, bf16 on mma.sync, split over the ring
// Per CTA: 16 heads of one sequence against tiles of 32 ring rows. A tile is the key AND the value of all heads, so it is
// fetched once (TMA, 128B-swizzled chunks of 64 columns into a ring of stages, by a warp of its own) and read twice from
// shared memory: S = Q K^T with the rows as the N operand, O += P C with the same rows transposed by ldmatrix. N is 32
// rows and M 16 heads, far below a tcgen05 tile. More heads are more CTAs, whose reads of the ring meet in L2.
//
// In S every warp takes an eighth of the columns, with its part of the queries in registers; the eight partial tiles meet in
// shared memory, where every warp does the softmax of two heads (lane = row); in O it takes its 64 columns. Two groups of
// eight warps work on alternate tiles of the same ring of stages: one computes while the other waits at its barrier, and
// enough tiles stay in flight. Each group leaves partial sums, which a second kernel puts together.
constexpr int LM_WARPS = 8;
constexpr int LM_GROUPS = 2;
constexpr int LM_THREADS = 32 * LM_WARPS * LM_GROUPS + 32;
constexpr int LM_KEYS = 32;
constexpr int LM_HEADS = 16;
constexpr int LM_SPITCH = 40;  // of score rows (fp32) and weight rows (bf16): conflict-free float2 stores and ldmatrix
constexpr int LM_MAX_STAGES = 6;
constexpr int LM_CHUNK = LM_KEYS * 128;  // bytes of [32 rows x 64 columns]
constexpr int LM_GROUP_BYTES = LM_HEADS * (LM_SPITCH * (LM_WARPS * 4 + 2) + 4);

__device__ __forceinline__ void lm_ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lm_ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ float lm_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// barrier of the eight warps of one group
__device__ __forceinline__ void lm_group_sync(int group) {
  asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "n"(32 * LM_WARPS) : "memory");
}
__device__ __forceinline__ void lm_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct LmParams {
  const __nv_bfloat16 *q_abs, *q;
  __nv_bfloat16* out;      // (heads, B, kvp)
  float* part_o;           // (n_part, B, heads, kvp), n_part = n_split · LM_GROUPS
  float* part_ml;          // (n_part, B, heads, 2)
  const int *slots, *start;
  int* status;
  int B, heads, dimp, rp, kvp, ring_len, n_split, stages;
  int chunks, ksteps;      // chunks of 64 and steps of 16 columns of a row
  float scale_log2;
};

// KW: steps of 16 columns per warp in the first product, NP: pairs of 8-column tiles per warp in the second
template <int KW, int NP>
__global__ void __launch_bounds__(LM_THREADS, 1)
latent_decode_mma_kernel(const __grid_constant__ CUtensorMap tmR, const LmParams p) {
  extern __shared__ __align__(1024) uint8_t lm_smem[];
  constexpr int HB = LM_HEADS;
  const int stage_bytes = p.chunks * LM_CHUNK;
  uint8_t* sk = lm_smem;
  const int tid = threadIdx.x, lane = tid & 31;
  const int group = (tid >> 5) / LM_WARPS, warp = (tid >> 5) % LM_WARPS;  // group LM_GROUPS: the producer
  // per group: [LM_WARPS][HB][LM_SPITCH] partial scores, [HB][LM_SPITCH] weights, [HB] rescale factors
  float* ss = reinterpret_cast<float*>(sk + p.stages * stage_bytes + (group % LM_GROUPS) * LM_GROUP_BYTES);
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(ss + LM_WARPS * HB * LM_SPITCH);
  float* sf = reinterpret_cast<float*>(sp + HB * LM_SPITCH);
  uint64_t* full = reinterpret_cast<uint64_t*>(sk + p.stages * stage_bytes + LM_GROUPS * LM_GROUP_BYTES);
  uint64_t* empty = full + LM_MAX_STAGES;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty + LM_MAX_STAGES);
  const int b = blockIdx.x, split = blockIdx.y, h0 = blockIdx.z * HB;
  const int lw = p.kvp + p.rp;
  const int nk = min(p.start[b] + 1, p.ring_len);
  const int nT = (nk + LM_KEYS - 1) / LM_KEYS;
  const int per = (nT + p.n_split - 1) / p.n_split;
  const int ta = split * per, tb = min(nT, ta + per);
  if (smem_u32(lm_smem) & 1023u) {
    if (tid == 0 && p.status) atomicCAS(p.status, 0, STATUS_TIMEOUT_MISC);
    return;
  }
  if (tid == 0) {
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], LM_WARPS);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  __syncthreads();
  if (group == LM_GROUPS) {
    // ------------------------------------------------------------ producer
    if (lane == 0) {
      tma_prefetch_desc(&tmR);
      const int row0 = p.slots[b] * p.ring_len;
      int stage = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int t = ta; t < tb; ++t) {
        if (!(ok = mbar_wait_bounded(&empty[stage], phase ^ 1, abort_flag, p.status, STATUS_TIMEOUT_EMPTY))) break;
        mbar_expect_tx(&full[stage], (uint32_t)stage_bytes);
        // rows beyond the last visible one belong to nobody or to the next slot: they are hidden below
        for (int c = 0; c < p.chunks; ++c) tma_load_2d(sk + stage * stage_bytes + c * LM_CHUNK, &tmR, &full[stage], 64 * c, row0 + t * LM_KEYS);
        if (++stage == p.stages) {
          stage = 0;
          phase ^= 1;
        }
      }
      if (!ok) {  // copies in flight get a bounded time to land before the shared memory is released
        const long long c0 = clock64();
        while (clock64() - c0 < 2000000LL) {
        }
      }
    }
    return;
  }
  float acc[2 * NP][4];
#pragma unroll
  for (int j = 0; j < 2 * NP; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  // this warp's columns of the queries as A operands: rows lane / 4 and + 8, columns (lane % 4) · 2 and + 8 of a step;
  // zero beyond the heads and the columns of a row
  const int k0 = warp * KW;
  uint32_t qf[KW][4];
#pragma unroll
  for (int i = 0; i < KW; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = h0 + (lane >> 2) + 8 * (e & 1), c = (k0 + i) * 16 + (lane & 3) * 2 + 8 * (e >> 1);
      qf[i][e] = 0u;
      if (h < p.heads && c < lw)
        qf[i][e] = *reinterpret_cast<const uint32_t*>(c < p.kvp ? p.q_abs + ((long long)h * p.B + b) * p.kvp + c
                                                                : p.q + ((long long)b * p.heads + h) * (p.dimp + p.rp) + p.dimp + c - p.kvp);
    }
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};  // heads 2 · warp, 2 · warp + 1; sums of this lane's rows
  const int n_pairs = (p.kvp + 15) / 16;
  // ldmatrix addresses within a stage: 16 ring rows x 16 columns per load, in the first product rows by columns, in the second
  // transposed; loads beyond the columns of a row meet zero queries or sums that are not kept, and read the first chunk
  uint32_t koff[KW], voff[NP];
  {
    const int kr = (lane & 7) + ((lane >> 4) << 3), vr = lane & 15;
#pragma unroll
    for (int i = 0; i < KW; ++i) {
      const int k = k0 + i < p.ksteps ? k0 + i : 0;
      koff[i] = (uint32_t)((k >> 2) * LM_CHUNK + kr * 128 + ((((k & 3) * 2 + ((lane >> 3) & 1)) ^ (kr & 7)) << 4));
    }
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int np = warp * NP + j < n_pairs ? warp * NP + j : 0;
      voff[j] = (uint32_t)((np >> 2) * LM_CHUNK + vr * 128 + ((((np & 3) * 2 + (lane >> 4)) ^ (vr & 7)) << 4));
    }
  }
  const uint32_t pa0 = smem_u32(sp + (lane & 15) * LM_SPITCH + (lane >> 4) * 8);
  float* const sd = ss + (warp * HB + (lane >> 2)) * LM_SPITCH + (lane & 3) * 2;
  const float* const sr = ss + warp * 2 * LM_SPITCH + lane;
  bool ok = true;
  int stage = group;  // at least LM_GROUPS + 1 stages
  uint32_t phase = 0;
  for (int t = ta + group; t < tb; t += LM_GROUPS) {
    // after a wait that ran out the tiles are worked on unseen: the status word tells, and the loop ends
    if (ok) ok = mbar_wait_bounded(&full[stage], phase, abort_flag, p.status, STATUS_TIMEOUT_FULL);
    const uint32_t kt = smem_u32(sk + stage * stage_bytes);
    {
      float s[LM_KEYS / 8][4];
#pragma unroll
      for (int i = 0; i < LM_KEYS / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
#pragma unroll
      for (int i = 0; i < KW; ++i) {
#pragma unroll
        for (int g = 0; g < LM_KEYS / 16; ++g) {
          uint32_t bb[4];
          lm_ldsm4(bb, kt + koff[i] + g * 16 * 128);
          lm_mma(s[2 * g], qf[i], bb[0], bb[1]);
          lm_mma(s[2 * g + 1], qf[i], bb[2], bb[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < LM_KEYS / 8; ++i) {
        *reinterpret_cast<float2*>(sd + 8 * i) = make_float2(s[i][0], s[i][1]);
        *reinterpret_cast<float2*>(sd + 8 * LM_SPITCH + 8 * i) = make_float2(s[i][2], s[i][3]);
      }
    }
    lm_group_sync(group);
    const bool seen = t * LM_KEYS + lane < nk;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = warp * 2 + i;
      float part[LM_WARPS];
#pragma unroll
      for (int g = 0; g < LM_WARPS; ++g) part[g] = sr[(g * HB + i) * LM_SPITCH];
      const float score = ((part[0] + part[1]) + (part[2] + part[3])) + ((part[4] + part[5]) + (part[6] + part[7]));
      const float x = seen ? score * p.scale_log2 : -INFINITY;
      const float mn = fmaxf(mx[i], warp_max(x));
      const float f = lm_exp2(mx[i] - mn), w = lm_exp2(x - mn);
      mx[i] = mn;
      sum[i] = fmaf(sum[i], f, w);
      sp[r * LM_SPITCH + lane] = __float2bfloat16_rn(w);
      if (lane == 0) sf[r] = f;
    }
    lm_group_sync(group);
    const float f0 = sf[lane >> 2], f1 = sf[(lane >> 2) + 8];
    if (__any_sync(0xffffffffu, f0 != 1.f || f1 != 1.f)) {
#pragma unroll
      for (int j = 0; j < 2 * NP; ++j) {
        acc[j][0] *= f0;
        acc[j][1] *= f0;
        acc[j][2] *= f1;
        acc[j][3] *= f1;
      }
    }
#pragma unroll
    for (int k = 0; k < LM_KEYS / 16; ++k) {
      uint32_t pa[4];
      lm_ldsm4(pa, pa0 + k * 32);
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        uint32_t v[4];
        lm_ldsm4t(v, kt + voff[j] + k * 16 * 128);
        lm_mma(acc[2 * j], pa, v[0], v[1]);
        lm_mma(acc[2 * j + 1], pa, v[2], v[3]);
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[stage]);
    stage += LM_GROUPS;
    if (stage >= p.stages) {
      stage -= p.stages;
      phase ^= 1;
    }
  }
  const long long part = ((long long)(split * LM_GROUPS + group) * p.B + b) * p.heads + h0;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = warp * 2 + i;
    const float l = warp_sum(sum[i]);
    if (lane == 0 && h0 + r < p.heads) *reinterpret_cast<float2*>(p.part_ml + (part + r) * 2) = make_float2(mx[i], l);
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = (lane >> 2) + 8 * e;
    if (h0 + r >= p.heads) continue;
#pragma unroll
    for (int j = 0; j < 2 * NP; ++j) {
      const int c = (warp * 2 * NP + j) * 8 + (lane & 3) * 2;
      if (c < p.kvp) *reinterpret_cast<float2*>(p.part_o + (part + r) * p.kvp + c) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
    }
  }
}

__global__ void __launch_bounds__(128)
latent_merge_kernel(const LmParams p) {
  __shared__ float wt[64];
  const int n_part = p.n_split * LM_GROUPS;
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31;
  const long long bh = (long long)b * p.heads + h, step = (long long)p.B * p.heads;
  if (threadIdx.x < 32) {  // at most 64 parts: two per lane
    float m[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = lane + 32 * i;
      const float2 v = s < n_part ? *reinterpret_cast<const float2*>(p.part_ml + (s * step + bh) * 2) : make_float2(-INFINITY, 0.f);
      m[i] = v.x;
      l[i] = v.y;
    }
    const float M = warp_max(fmaxf(m[0], m[1]));
    float f[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) f[i] = m[i] == -INFINITY ? 0.f : exp2f(m[i] - M);
    const float inv = 1.f / warp_sum(f[0] * l[0] + f[1] * l[1]);
    wt[lane] = f[0] * inv;
    wt[lane + 32] = f[1] * inv;
  }
  __syncthreads();
  for (int c = threadIdx.x * 4; c < p.kvp; c += 512) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < n_part; ++s) {
      const float4 v = *reinterpret_cast<const float4*>(p.part_o + (s * step + bh) * p.kvp + c);
      const float w = wt[s];  // 0 for a part that saw no row (its sums are zero)
      o.x = fmaf(w, v.x, o.x);
      o.y = fmaf(w, v.y, o.y);
      o.z = fmaf(w, v.z, o.z);
      o.w = fmaf(w, v.w, o.w);
    }
    *reinterpret_cast<uint2*>(p.out + ((long long)h * p.B + b) * p.kvp + c) = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
  }
}

static size_t lm_smem_bytes(int chunks, int stages) {
  return (size_t)stages * chunks * LM_CHUNK + LM_GROUPS * LM_GROUP_BYTES + 2 * LM_MAX_STAGES * 8 + 16;
}

struct LmPlan {
  int chunks, ksteps, stages, n_split;
};
static LmPlan lm_plan(int B, int heads, int kvp, int rp, int ring_len) {
  LmPlan pl;
  pl.chunks = (kvp + rp + 63) / 64;
  pl.ksteps = (kvp + rp + 15) / 16;
  pl.stages = 0;
  for (int st = LM_MAX_STAGES; st >= LM_GROUPS + 1 && !pl.stages; --st)
    if (lm_smem_bytes(pl.chunks, st) <= 232448) pl.stages = st;
  const long long ctas = (long long)B * ((heads + LM_HEADS - 1) / LM_HEADS);
  const int tiles = (ring_len + LM_KEYS - 1) / LM_KEYS;
  long long n = 148 / ctas;  // one CTA per SM: a second, partly filled wave would cost as much as the first
  if (n > (tiles + 7) / 8) n = (tiles + 7) / 8;
  if (n > 64 / LM_GROUPS) n = 64 / LM_GROUPS;
  pl.n_split = n < 1 ? 1 : (int)n;
  return pl;
}

template <int KW, int NP>
static int lm_launch(const CUtensorMap& tm, const LmParams& p, cudaStream_t s) {
  const size_t smem = lm_smem_bytes(p.chunks, p.stages);
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(latent_decode_mma_kernel<KW, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
  const dim3 grid(p.B, p.n_split, (p.heads + LM_HEADS - 1) / LM_HEADS);
  latent_decode_mma_kernel<KW, NP><<<grid, LM_THREADS, smem, s>>>(tm, p);
  latent_merge_kernel<<<dim3(p.heads, p.B), 128, 0, s>>>(p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

}  // namespace kvb

#define KVB_LATENT_TYPES(dtype, ...)                          \
  switch (dtype) {                                            \
    case 0: { using T = float; __VA_ARGS__; break; }          \
    case 1: { using T = __nv_bfloat16; __VA_ARGS__; break; }  \
    default: return KVB_ERR_ARG;                              \
  }

extern "C" int kvb_latent_prep(const void* qkv, long long ld, const float* norm_w, const float* freq, void* q, void* latent, void* ring,
                               const int* slots, const int* start, const int* count, int B, int T_, int P, int ring_len, int heads,
                               int dim, int dimp, int rot, int rot_dims, int rp, int kv_rank, int kvp, float eps, int dtype,
                               void* stream) {
  if (B <= 0 || T_ <= 0 || heads <= 0 || dimp < dim || rp < rot || kvp < kv_rank || rot_dims > rot || rot_dims % 2 || B > 65535)
    return KVB_ERR_ARG;
  if (ring && ring_len <= 0) return KVB_ERR_ARG;
  if ((dimp | rp | kvp) % 8) return KVB_ERR_ALIGN;
  kvb::LpParams p;
  p.ld = ld; p.norm_w = norm_w; p.freq = freq; p.slots = slots; p.start = start; p.count = count;
  p.T = T_; p.P = P; p.ring_len = ring_len; p.heads = heads; p.dim = dim; p.dimp = dimp; p.rot = rot; p.rot_dims = rot_dims; p.rp = rp;
  p.kv_rank = kv_rank; p.kvp = kvp; p.eps = eps;
  KVB_LATENT_TYPES(dtype, return kvb::lp_launch<T>(qkv, q, latent, ring, p, B, (cudaStream_t)stream));
}

extern "C" int kvb_ring_gather(const void* ring, void* latent, const int* slots, const int* start, int B, int T_, int P, int ring_len,
                               int lw, int dtype, void* stream) {
  if (P <= 0) return KVB_OK;
  if (B <= 0 || B > 65535 || ring_len <= 0 || lw % 8 || (dtype != 0 && dtype != 1)) return KVB_ERR_ARG;
  kvb::ring_gather_kernel<<<dim3((P + kvb::LR_WARPS - 1) / kvb::LR_WARPS, B), kvb::LR_WARPS * 32, 0, (cudaStream_t)stream>>>(
      (const uint4*)ring, (uint4*)latent, slots, start, T_, P, ring_len, lw / (dtype == 0 ? 4 : 8));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_latent_attend(const void* q, const void* kv, const void* latent, void* out, const int* start, int B, int T_, int P,
                                 int heads, int dimp, int rp, int kvp, int vdp, int window, float scale, int dtype, void* stream) {
  if (B <= 0 || T_ <= 0 || B > 65535 || heads > 65535 || (dimp | rp) & 1) return KVB_ERR_ARG;
  if (vdp > 32 * kvb::LA_MAX_V) return KVB_ERR_TOO_LARGE;
  const size_t smem = kvb::LA_WARPS * (dimp + rp) * sizeof(float);
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  const dim3 grid((T_ + kvb::LA_WARPS - 1) / kvb::LA_WARPS, heads, B);
  KVB_LATENT_TYPES(dtype, (kvb::latent_attend_simple_kernel<T><<<grid, kvb::LA_WARPS * 32, smem, (cudaStream_t)stream>>>(
      (const T*)q, (const T*)kv, (const T*)latent, (T*)out, start, T_, P, heads, dimp, rp, kvp, vdp, window, scale)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" long long kvb_latent_decode_scratch_bytes(int B, int heads, int kvp, int rp, int ring_len) {
  const int n = kvb::lm_plan(B, heads, kvp, rp, ring_len).n_split;
  return (long long)n * kvb::LM_GROUPS * B * heads * (kvp + 2) * 4;
}

extern "C" int kvb_latent_decode(const void* q_abs, const void* q, const void* ring, void* out, void* scratch, const int* slots,
                                 const int* start, int B, int n_slots, int heads, int dimp, int rp, int kvp, int ring_len,
                                 float scale, int dtype, int simple, int* status, void* stream) {
  using namespace kvb;
  if (B <= 0 || heads <= 0 || ring_len <= 0 || B > 65535) return KVB_ERR_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  LmParams p;
  const LmPlan pl = lm_plan(B, heads, kvp, rp, ring_len);
  p.chunks = pl.chunks; p.ksteps = pl.ksteps; p.stages = pl.stages; p.n_split = pl.n_split;
  if (dtype == 1 && !simple && kvp % 8 == 0 && rp % 8 == 0 && dimp % 8 == 0 && kvp <= 512 && p.stages > 0 && n_slots > 0 &&
      p.ksteps <= 40) {
    CUtensorMap tm;
    const uint64_t lw = kvp + rp, dims[2] = {lw, (uint64_t)n_slots * ring_len}, st[1] = {lw};
    const uint32_t box[2] = {64, LM_KEYS};
    const int rc = tmap_bf16(&tm, ring, 2, dims, st, box);
    if (rc) return rc;
    p.q_abs = (const __nv_bfloat16*)q_abs; p.q = (const __nv_bfloat16*)q;
    p.out = (__nv_bfloat16*)out; p.slots = slots; p.start = start;
    p.B = B; p.heads = heads; p.dimp = dimp; p.rp = rp; p.kvp = kvp; p.ring_len = ring_len;
    p.part_o = (float*)scratch;
    p.part_ml = p.part_o + (long long)p.n_split * LM_GROUPS * B * heads * kvp;
    p.scale_log2 = scale * 1.4426950408889634f;
    p.status = status;
    if (kvp <= 128 && p.ksteps <= 16) return lm_launch<2, 1>(tm, p, s);
    if (kvp <= 256 && p.ksteps <= 24) return lm_launch<3, 2>(tm, p, s);
    return lm_launch<5, 4>(tm, p, s);
  }
  if (kvp > 32 * LD_MAX_C) return KVB_ERR_TOO_LARGE;
  const size_t smem = ((size_t)kvp + rp + 4 * kvp + 8) * sizeof(float);
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  KVB_LATENT_TYPES(dtype, (latent_decode_simple_kernel<T><<<dim3(heads, B), 128, smem, s>>>(
      (const T*)q_abs, (const T*)q, (const T*)ring, (T*)out, slots, start, B, heads, dimp, rp, kvp, ring_len, scale)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
