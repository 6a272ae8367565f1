// Latent attention: queries of H heads against one latent per token (plus one rotated key part that the heads share).
//
//   prep    splits the joint projection, norms the latent, rotates the rotary parts (angles in fp32, computed once per
//           token), writes padded query and latent rows; a single-token pass writes its latent row straight into the ring;
//   ring    a layer that sees a window of W tokens keeps W latents per sequence: position p lives in slot p mod length;
//   attend  several new tokens: keys and values of the window before the pass and of the pass itself are expanded from
//           the latents by a matrix product and swept with an online softmax (here on CUDA cores, for fp32 and for shapes the
//           tcgen05 kernel of latent_sm100.cu does not take);
//   decode  one new token per sequence stays in latent space: W_uk is folded into the query and W_uv into the output, so
//           the ring is read once for all heads and serves as key and value.
#include "common.cuh"
#include "kvb200_layers.h"

namespace kvb {

// ------------------------------------------------------------------------------------------------ prep
// One warp per unit of a token: unit h < heads is a query head, unit `heads` the latent row. A CTA has 8 units of one token and
// computes the token's angles once. V elements per access (16 bytes, or 1 when the sizes do not divide).
constexpr int LP_WARPS = 8;

template <typename T, int V>
struct alignas(sizeof(T) * V) LpVec {
  T v[V];
};

struct LpParams {
  long long ld;
  const float *norm_w, *freq;
  const int *slots, *start, *count;
  int T, P, ring_len, heads, dim, dimp, rot, rot_dims, rp, kv_rank, kvp;
  float eps;
};

// the rotary part x (rot elements, the first rot_dims rotated) to dst, zero up to rp
template <typename T, int V>
__device__ __forceinline__ void lp_rotate(const T* __restrict__ x, T* __restrict__ dst, const float* cs, const float* sn, const LpParams& p,
                                          int lane) {
  using Vec = LpVec<T, V>;
  const int half = p.rot_dims / 2;
  for (int i = lane * V; i < half; i += 32 * V) {
    const Vec a = *reinterpret_cast<const Vec*>(x + i), b = *reinterpret_cast<const Vec*>(x + half + i);
    Vec c, d;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float u = to_f32(a.v[e]), v = to_f32(b.v[e]);
      c.v[e] = from_f32<T>(u * cs[i + e] - v * sn[i + e]);
      d.v[e] = from_f32<T>(v * cs[i + e] + u * sn[i + e]);
    }
    *reinterpret_cast<Vec*>(dst + i) = c;
    *reinterpret_cast<Vec*>(dst + half + i) = d;
  }
  for (int i = p.rot_dims + lane; i < p.rp; i += 32) dst[i] = i < p.rot ? x[i] : from_f32<T>(0.f);
}

template <typename T, int V>
__global__ void __launch_bounds__(LP_WARPS * 32)
latent_prep_kernel(const T* __restrict__ qkv, T* __restrict__ q, T* __restrict__ latent, T* __restrict__ ring, const LpParams p) {
  using Vec = LpVec<T, V>;
  extern __shared__ float sm[];  // cos | sin (rot_dims / 2 each)
  const int t = blockIdx.x, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int unit = blockIdx.y * LP_WARPS + warp;
  const long long n = (long long)b * p.T + t;
  const int pos = p.start[b] + t;
  const int half = p.rot_dims / 2;
  float *cs = sm, *sn = sm + half;
  for (int i = threadIdx.x; i < half; i += LP_WARPS * 32) sincosf((float)pos * p.freq[i], &sn[i], &cs[i]);
  __syncthreads();
  const T* src = qkv + n * p.ld;
  if (unit < p.heads) {
    const T* x = src + unit * (p.dim + p.rot);
    T* dst = q + (n * p.heads + unit) * (p.dimp + p.rp);
    for (int i = lane * V; i < p.dim; i += 32 * V) *reinterpret_cast<Vec*>(dst + i) = *reinterpret_cast<const Vec*>(x + i);
    for (int i = p.dim + lane; i < p.dimp; i += 32) dst[i] = from_f32<T>(0.f);
    lp_rotate<T, V>(x + p.dim, dst + p.dimp, cs, sn, p, lane);
    return;
  }
  if (unit > p.heads) return;
  T* dst;
  if (ring) {
    if (p.count[b] <= t) return;  // padding never reaches the ring
    dst = ring + ((long long)p.slots[b] * p.ring_len + pos % p.ring_len) * (p.kvp + p.rp);
  } else {
    dst = latent + ((long long)b * (p.P + p.T) + p.P + t) * (p.kvp + p.rp);
  }
  const T* c = src + p.heads * (p.dim + p.rot);
  float ss = 0.f;
  for (int i = lane * V; i < p.kv_rank; i += 32 * V) {
    const Vec a = *reinterpret_cast<const Vec*>(c + i);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(to_f32(a.v[e]), to_f32(a.v[e]), ss);
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)p.kv_rank + p.eps);
  for (int i = lane * V; i < p.kv_rank; i += 32 * V) {
    Vec a = *reinterpret_cast<const Vec*>(c + i);
#pragma unroll
    for (int e = 0; e < V; ++e) a.v[e] = from_f32<T>(to_f32(a.v[e]) * r * p.norm_w[i + e]);
    *reinterpret_cast<Vec*>(dst + i) = a;
  }
  for (int i = p.kv_rank + lane; i < p.kvp; i += 32) dst[i] = from_f32<T>(0.f);
  lp_rotate<T, V>(c + p.kv_rank, dst + p.kvp, cs, sn, p, lane);
}

template <typename T>
static int lp_launch(const void* qkv, void* q, void* latent, void* ring, const LpParams& p, int B, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const dim3 grid(p.T, (p.heads + LP_WARPS) / LP_WARPS, B);
  const size_t smem = p.rot_dims * sizeof(float) + 8;
  if (((p.dim | p.rot | p.kv_rank | (p.rot_dims / 2)) % V) == 0 && p.ld % V == 0)
    latent_prep_kernel<T, V><<<grid, LP_WARPS * 32, smem, s>>>((const T*)qkv, (T*)q, (T*)latent, (T*)ring, p);
  else
    latent_prep_kernel<T, 1><<<grid, LP_WARPS * 32, smem, s>>>((const T*)qkv, (T*)q, (T*)latent, (T*)ring, p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
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

__global__ void __launch_bounds__(LR_WARPS * 32)
ring_append_kernel(const uint4* __restrict__ latent, uint4* __restrict__ ring, const int* __restrict__ slots, const int* __restrict__ start,
                   const int* __restrict__ count, int Tn, int P, int ring_len, int units) {
  const int i0 = blockIdx.x * LR_WARPS + (threadIdx.x >> 5), b = blockIdx.y;
  const int t = count[b] - 1 - i0;  // newest first
  if (t < 0 || i0 >= ring_len) return;
  const uint4* src = latent + ((long long)b * (P + Tn) + P + t) * units;
  uint4* dst = ring + ((long long)slots[b] * ring_len + (start[b] + t) % ring_len) * units;
  for (int i = threadIdx.x & 31; i < units; i += 32) dst[i] = src[i];
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
// Per CTA: 16 · MT heads of one sequence against tiles of 32 ring rows. A tile is the key AND the value of all heads, so it is
// fetched once (one bulk copy per row into a ring of stages) and read twice from shared memory: S = Q K^T with the rows as
// the N operand, O += P C with the same rows transposed by ldmatrix. N is 32 rows and M 16 or 32 heads, far below a
// tcgen05 tile, and the kernel is bound by the read of the ring.
//
// Warps 0..3 and 4..7 take the two halves of the features in S (8 rows each); after one barrier every warp has the whole S tile
// in the layout of the A operand of the second product, so each keeps maximum and sum of all heads in registers
// and no second exchange is needed. The barrier of tile t also says that everybody is done with tile t − 1: its
// stage is refilled then.
constexpr int LM_THREADS = 256;
constexpr int LM_KEYS = 32;
constexpr int LM_SPITCH = 40;
constexpr int LM_MAX_STAGES = 6;

__device__ __forceinline__ void lm_ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lm_ldsm2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lm_ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lm_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct LmParams {
  const __nv_bfloat16 *q_abs, *q, *ring;
  __nv_bfloat16* out;      // (heads, B, kvp)
  float* part_o;           // (n_split, B, heads, kvp)
  float* part_ml;          // (n_split, B, heads, 2)
  const int *slots, *start;
  int* status;
  int B, heads, dimp, rp, kvp, ring_len, n_split, stages;
  int kv16, ls;            // latent columns rounded up to 16; row pitch in shared memory (elements)
  float scale_log2;
};

// MT: tiles of 16 heads; NP: pairs of 8-column tiles per warp in the second product
template <int MT, int NP>
__global__ void __launch_bounds__(LM_THREADS, 1)
latent_decode_mma_kernel(const LmParams p) {
  extern __shared__ __align__(128) uint8_t lm_smem[];
  constexpr int HB = 16 * MT;
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(lm_smem);
  __nv_bfloat16* sk = sq + HB * p.ls;
  float* ss = reinterpret_cast<float*>(sk + p.stages * LM_KEYS * p.ls);  // [2 tiles][2 halves][HB][LM_SPITCH]
  uint64_t* full = reinterpret_cast<uint64_t*>(ss + 4 * HB * LM_SPITCH);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(full + LM_MAX_STAGES);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.x, split = blockIdx.y, h0 = blockIdx.z * HB;
  const int lw = p.kvp + p.rp;
  const int nk = min(p.start[b] + 1, p.ring_len);
  const int nT = (nk + LM_KEYS - 1) / LM_KEYS;
  const int per = (nT + p.n_split - 1) / p.n_split;
  const int ta = split * per, tb = min(nT, ta + per);
  const __nv_bfloat16* base = p.ring + (long long)p.slots[b] * p.ring_len * lw;
  // zero query rows and the padding columns that no copy writes
  for (int i = tid; i < (HB + p.stages * LM_KEYS) * p.ls / 8; i += LM_THREADS) reinterpret_cast<uint4*>(lm_smem)[i] = make_uint4(0, 0, 0, 0);
  if (tid == 0) {
    for (int i = 0; i < p.stages; ++i) mbar_init(&full[i], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  fence_proxy_async_smem();
  __syncthreads();
  auto load_tile = [&](int t, int stage) {  // warp 0: one row per lane
    __nv_bfloat16* dst = sk + (stage * LM_KEYS + lane) * p.ls;
    const int rows = min(LM_KEYS, nk - t * LM_KEYS);
    const __nv_bfloat16* src = base + (long long)(t * LM_KEYS + lane) * lw;
    if (lane == 0) mbar_expect_tx(&full[stage], (uint32_t)(rows * lw * 2));
    __syncwarp();
    if (lane < rows) {
      if (p.kv16 == p.kvp) {
        bulk_load(dst, src, (uint32_t)(lw * 2), &full[stage]);
      } else {
        bulk_load(dst, src, (uint32_t)(p.kvp * 2), &full[stage]);
        bulk_load(dst + p.kv16, src + p.kvp, (uint32_t)(p.rp * 2), &full[stage]);
      }
    }
  };
  if (warp == 0)
    for (int i = 0; i < p.stages && ta + i < tb; ++i) load_tile(ta + i, i);
  const int ku = p.kvp / 8, lu = lw / 8;
  for (int i = tid; i < HB * lu; i += LM_THREADS) {
    const int h = i / lu, u = i - h * lu;
    if (h0 + h < p.heads) {
      const __nv_bfloat16* src = u < ku ? p.q_abs + ((long long)(h0 + h) * p.B + b) * p.kvp + u * 8
                                        : p.q + ((long long)b * p.heads + h0 + h) * (p.dimp + p.rp) + p.dimp + (u - ku) * 8;
      *reinterpret_cast<uint4*>(sq + h * p.ls + (u < ku ? u * 8 : p.kv16 + (u - ku) * 8)) = *reinterpret_cast<const uint4*>(src);
    }
  }
  float acc[MT][2 * NP][4];
  float mx[MT][2], sum[MT][2];
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    mx[m][0] = mx[m][1] = -INFINITY;
    sum[m][0] = sum[m][1] = 0.f;
#pragma unroll
    for (int j = 0; j < 2 * NP; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][j][e] = 0.f;
  }
  __syncthreads();
  const int ksteps = (p.ls - 8) / 16;
  const int half = warp >> 2, k_lo = half ? (ksteps + 1) / 2 : 0, k_hi = half ? ksteps : (ksteps + 1) / 2;
  const int key0 = (warp & 3) * 8;
  const int n_pairs = p.kv16 / 16;
  bool ok = true;
  int stage = 0;
  uint32_t phase = 0;
  for (int t = ta; t < tb; ++t) {
    // after a wait that ran out the tiles are worked on unseen: the status word tells, and the loop ends
    if (ok) ok = mbar_wait_bounded(&full[stage], phase, abort_flag, p.status, STATUS_TIMEOUT_FULL);
    const __nv_bfloat16* kt = sk + stage * LM_KEYS * p.ls;
    {
      float s[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[m][i][e] = 0.f;
      const uint32_t qa = smem_u32(sq + (lane & 15) * p.ls + (lane >> 4) * 8);
      const uint32_t kb = smem_u32(kt + (key0 + (lane & 7)) * p.ls + (lane >> 3) * 8);
      int k = k_lo;
#pragma unroll 2
      for (; k + 1 < k_hi; k += 2) {
        uint32_t bb[4];
        lm_ldsm4(bb, kb + k * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a[4];
          lm_ldsm4(a, qa + m * 16 * p.ls * 2 + k * 32);
          lm_mma(s[m][0], a, bb[0], bb[1]);
          lm_ldsm4(a, qa + m * 16 * p.ls * 2 + k * 32 + 32);
          lm_mma(s[m][1], a, bb[2], bb[3]);
        }
      }
      if (k < k_hi) {
        uint32_t b0, b1;
        lm_ldsm2(b0, b1, smem_u32(kt + (key0 + (lane & 7)) * p.ls + ((lane >> 3) & 1) * 8) + k * 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a[4];
          lm_ldsm4(a, qa + m * 16 * p.ls * 2 + k * 32);
          lm_mma(s[m][0], a, b0, b1);
        }
      }
      float* sd = ss + ((t & 1) * 2 + half) * HB * LM_SPITCH;
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const int r = m * 16 + (lane >> 2), c = key0 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(sd + r * LM_SPITCH + c) = make_float2(s[m][0][0] + s[m][1][0], s[m][0][1] + s[m][1][1]);
        *reinterpret_cast<float2*>(sd + (r + 8) * LM_SPITCH + c) = make_float2(s[m][0][2] + s[m][1][2], s[m][0][3] + s[m][1][3]);
      }
    }
    __syncthreads();
    if (warp == 0 && t > ta && t - 1 + p.stages < tb) load_tile(t - 1 + p.stages, stage == 0 ? p.stages - 1 : stage - 1);
    const int left = nk - t * LM_KEYS;
    const float* s0 = ss + (t & 1) * 2 * HB * LM_SPITCH;
    const float* s1 = s0 + HB * LM_SPITCH;
    uint32_t pa[MT][LM_KEYS / 16][4];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {  // rows lane / 4 and lane / 4 + 8
        const int o = (m * 16 + (lane >> 2) + 8 * e) * LM_SPITCH + (lane & 3) * 2;
        float x[LM_KEYS / 4];
        float mn = mx[m][e];
#pragma unroll
        for (int i = 0; i < LM_KEYS / 8; ++i) {
          const float2 u = *reinterpret_cast<const float2*>(s0 + o + 8 * i), v = *reinterpret_cast<const float2*>(s1 + o + 8 * i);
          const int c = (lane & 3) * 2 + 8 * i;
          x[2 * i] = c < left ? (u.x + v.x) * p.scale_log2 : -INFINITY;
          x[2 * i + 1] = c + 1 < left ? (u.y + v.y) * p.scale_log2 : -INFINITY;
          mn = fmax3(mn, x[2 * i], x[2 * i + 1]);
        }
        mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, 1));
        mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, 2));
        const float f = exp2f(mx[m][e] - mn);
        mx[m][e] = mn;
        float l = 0.f;
#pragma unroll
        for (int i = 0; i < LM_KEYS / 4; ++i) {
          x[i] = exp2f(x[i] - mn);
          l += x[i];
        }
        sum[m][e] = sum[m][e] * f + l;  // this lane's columns; the quad is added up at the end
#pragma unroll
        for (int i = 0; i < LM_KEYS / 16; ++i) {
          pa[m][i][e] = pack_bf16x2(x[4 * i], x[4 * i + 1]);
          pa[m][i][2 + e] = pack_bf16x2(x[4 * i + 2], x[4 * i + 3]);
        }
#pragma unroll
        for (int j = 0; j < 2 * NP; ++j) {
          acc[m][j][2 * e] *= f;
          acc[m][j][2 * e + 1] *= f;
        }
      }
    }
#pragma unroll
    for (int k = 0; k < LM_KEYS / 16; ++k) {
      const uint32_t vb = smem_u32(kt + (k * 16 + (lane & 15)) * p.ls + (lane >> 4) * 8);
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int np = warp * NP + j;
        if (np < n_pairs) {
          uint32_t v[4];
          lm_ldsm4t(v, vb + np * 32);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            lm_mma(acc[m][2 * j], pa[m][k], v[0], v[1]);
            lm_mma(acc[m][2 * j + 1], pa[m][k], v[2], v[3]);
          }
        }
      }
    }
    if (++stage == p.stages) {
      stage = 0;
      phase ^= 1;
    }
  }
  const bool direct = p.n_split == 1;
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float l = sum[m][e];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      const int r = m * 16 + (lane >> 2) + 8 * e, h = h0 + r;
      if (h >= p.heads) continue;
      const float inv = direct ? 1.f / l : 1.f;
#pragma unroll
      for (int j = 0; j < 2 * NP; ++j) {
        const int c = (warp * 2 * NP + j) * 8 + (lane & 3) * 2;
        if (c >= p.kvp) continue;
        if (direct)
          *reinterpret_cast<uint32_t*>(p.out + ((long long)h * p.B + b) * p.kvp + c) =
              pack_bf16x2(acc[m][j][2 * e] * inv, acc[m][j][2 * e + 1] * inv);
        else
          *reinterpret_cast<float2*>(p.part_o + (((long long)split * p.B + b) * p.heads + h) * p.kvp + c) =
              make_float2(acc[m][j][2 * e], acc[m][j][2 * e + 1]);
      }
      if (!direct && warp == 0 && (lane & 3) == 0) {
        float* ml = p.part_ml + (((long long)split * p.B + b) * p.heads + h) * 2;
        ml[0] = mx[m][e];
        ml[1] = l;
      }
    }
  }
  if (!ok) {  // copies in flight get a bounded time to land before the shared memory is released
    const long long c0 = clock64();
    while (clock64() - c0 < 2000000LL) {
    }
  }
}

__global__ void __launch_bounds__(128)
latent_merge_kernel(const LmParams p) {
  const int h = blockIdx.x, b = blockIdx.y;
  const long long bh = (long long)b * p.heads + h, step = (long long)p.B * p.heads;
  float M = -INFINITY;
  for (int s = 0; s < p.n_split; ++s) M = fmaxf(M, p.part_ml[(s * step + bh) * 2]);
  float L = 0.f;
  for (int s = 0; s < p.n_split; ++s) {
    const float m = p.part_ml[(s * step + bh) * 2];
    if (m != -INFINITY) L += p.part_ml[(s * step + bh) * 2 + 1] * exp2f(m - M);
  }
  const float inv = 1.f / L;
  for (int c = threadIdx.x; c < p.kvp; c += 128) {
    float o = 0.f;
    for (int s = 0; s < p.n_split; ++s) {
      const float m = p.part_ml[(s * step + bh) * 2];
      if (m != -INFINITY) o = fmaf(p.part_o[(s * step + bh) * p.kvp + c], exp2f(m - M), o);
    }
    p.out[((long long)h * p.B + b) * p.kvp + c] = __float2bfloat16_rn(o * inv);
  }
}

static int lm_splits(int B, int heads, int ring_len) {
  const int hb = heads > 16 ? 32 : 16;
  const long long ctas = (long long)B * ((heads + hb - 1) / hb);
  const int tiles = (ring_len + LM_KEYS - 1) / LM_KEYS;
  long long n = 148 / ctas;  // one CTA per SM: a second, partly filled wave would cost as much as the first
  if (n > (tiles + 3) / 4) n = (tiles + 3) / 4;
  if (n > 64) n = 64;
  return n < 1 ? 1 : (int)n;
}

static size_t lm_smem_bytes(int mt, int ls, int stages) {
  const int hb = 16 * mt;
  return (size_t)(hb + stages * LM_KEYS) * ls * 2 + (size_t)4 * hb * LM_SPITCH * 4 + LM_MAX_STAGES * 8 + 16;
}

static int lm_stages(int mt, int ls) {
  for (int st = LM_MAX_STAGES; st >= 2; --st)
    if (lm_smem_bytes(mt, ls, st) <= 232448) return st;
  return 0;
}

template <int MT, int NP>
static int lm_launch(const LmParams& p, cudaStream_t s) {
  const size_t smem = lm_smem_bytes(MT, p.ls, p.stages);
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(latent_decode_mma_kernel<MT, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
  const dim3 grid(p.B, p.n_split, (p.heads + 16 * MT - 1) / (16 * MT));
  latent_decode_mma_kernel<MT, NP><<<grid, LM_THREADS, smem, s>>>(p);
  if (p.n_split > 1) latent_merge_kernel<<<dim3(p.heads, p.B), 128, 0, s>>>(p);
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
  if (ring && (T_ != 1 || ring_len <= 0)) return KVB_ERR_ARG;
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

extern "C" int kvb_ring_append(const void* latent, void* ring, const int* slots, const int* start, const int* count, int B, int T_,
                               int P, int ring_len, int lw, int dtype, void* stream) {
  if (B <= 0 || T_ <= 0 || B > 65535 || ring_len <= 0 || lw % 8 || (dtype != 0 && dtype != 1)) return KVB_ERR_ARG;
  const int rows = T_ < ring_len ? T_ : ring_len;
  kvb::ring_append_kernel<<<dim3((rows + kvb::LR_WARPS - 1) / kvb::LR_WARPS, B), kvb::LR_WARPS * 32, 0, (cudaStream_t)stream>>>(
      (const uint4*)latent, (uint4*)ring, slots, start, count, T_, P, ring_len, lw / (dtype == 0 ? 4 : 8));
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

extern "C" long long kvb_latent_decode_scratch_bytes(int B, int heads, int kvp, int ring_len) {
  const int n = kvb::lm_splits(B, heads, ring_len);
  return n == 1 ? 16 : (long long)n * B * heads * (kvp + 2) * 4;
}

extern "C" int kvb_latent_decode(const void* q_abs, const void* q, const void* ring, void* out, void* scratch, const int* slots,
                                 const int* start, int B, int heads, int dimp, int rp, int kvp, int ring_len, float scale, int dtype,
                                 int simple, int* status, void* stream) {
  using namespace kvb;
  if (B <= 0 || heads <= 0 || ring_len <= 0 || B > 65535) return KVB_ERR_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  LmParams p;
  p.kv16 = (kvp + 15) / 16 * 16;
  p.ls = p.kv16 + (rp + 15) / 16 * 16 + 8;
  const int mt = heads > 16 ? 2 : 1;
  p.stages = lm_stages(mt, p.ls);
  if (dtype == 1 && !simple && kvp % 8 == 0 && rp % 8 == 0 && dimp % 8 == 0 && kvp <= 512 && p.stages > 0) {
    p.q_abs = (const __nv_bfloat16*)q_abs; p.q = (const __nv_bfloat16*)q; p.ring = (const __nv_bfloat16*)ring;
    p.out = (__nv_bfloat16*)out; p.slots = slots; p.start = start;
    p.B = B; p.heads = heads; p.dimp = dimp; p.rp = rp; p.kvp = kvp; p.ring_len = ring_len;
    p.n_split = lm_splits(B, heads, ring_len);
    p.part_o = (float*)scratch;
    p.part_ml = p.part_o + (long long)p.n_split * B * heads * kvp;
    p.scale_log2 = scale * 1.4426950408889634f;
    p.status = status;
    const int np = (p.kv16 / 16 + 7) / 8;
    if (mt == 1) return np <= 1 ? lm_launch<1, 1>(p, s) : (np <= 2 ? lm_launch<1, 2>(p, s) : lm_launch<1, 4>(p, s));
    return np <= 1 ? lm_launch<2, 1>(p, s) : (np <= 2 ? lm_launch<2, 2>(p, s) : lm_launch<2, 4>(p, s));
  }
  if (kvp > 32 * LD_MAX_C) return KVB_ERR_TOO_LARGE;
  const size_t smem = ((size_t)kvp + rp + 4 * kvp + 8) * sizeof(float);
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  KVB_LATENT_TYPES(dtype, (latent_decode_simple_kernel<T><<<dim3(heads, B), 128, smem, s>>>(
      (const T*)q_abs, (const T*)q, (const T*)ring, (T*)out, slots, start, B, heads, dimp, rp, kvp, ring_len, scale)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
