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
constexpr int LP_THREADS = 128;

template <typename T>
__global__ void __launch_bounds__(LP_THREADS)
latent_prep_kernel(const T* __restrict__ qkv, long long ld, const float* __restrict__ norm_w, const float* __restrict__ freq,
                   T* __restrict__ q, T* __restrict__ latent, T* __restrict__ ring, const int* __restrict__ slots,
                   const int* __restrict__ start, const int* __restrict__ count, int Tn, int P, int ring_len, int heads, int dim,
                   int dimp, int rot, int rot_dims, int rp, int kv_rank, int kvp, float eps) {
  extern __shared__ float sm[];  // cos | sin (rot_dims / 2 each)
  __shared__ float red[LP_THREADS / 32];
  const int t = blockIdx.x, b = blockIdx.y;
  const long long n = (long long)b * Tn + t;
  const int pos = start[b] + t;
  const int half = rot_dims / 2;
  float *cs = sm, *sn = sm + half;
  for (int i = threadIdx.x; i < half; i += LP_THREADS) {
    const float a = (float)pos * freq[i];
    sincosf(a, &sn[i], &cs[i]);
  }
  const T* src = qkv + n * ld;
  const T* c = src + heads * (dim + rot);
  float ss = 0.f;
  for (int i = threadIdx.x; i < kv_rank; i += LP_THREADS) {
    const float v = to_f32(c[i]);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < LP_THREADS / 32; ++i) ss += red[i];
  const float r = 1.f / sqrtf(ss / (float)kv_rank + eps);
  const int lw = kvp + rp;
  T* dst = nullptr;
  if (ring) {
    if (count[b] > t) dst = ring + ((long long)slots[b] * ring_len + pos % ring_len) * lw;
  } else {
    dst = latent + ((long long)b * (P + Tn) + P + t) * lw;
  }
  // element i of a rotary part
  auto rotated = [&](const T* x, int i) {
    if (i >= rot_dims) return to_f32(x[i]);
    const int k = i < half ? i : i - half;
    const float u = to_f32(x[k]), v = to_f32(x[k + half]);
    return i < half ? u * cs[k] - v * sn[k] : v * cs[k] + u * sn[k];
  };
  if (dst) {
    for (int i = threadIdx.x; i < lw; i += LP_THREADS) {
      float v = 0.f;
      if (i < kv_rank) v = to_f32(c[i]) * r * norm_w[i];
      else if (i >= kvp && i - kvp < rot) v = rotated(c + kv_rank, i - kvp);
      dst[i] = from_f32<T>(v);
    }
  }
  const int dq = dimp + rp;
  T* qd = q + n * heads * dq;
  for (int i = threadIdx.x; i < heads * dq; i += LP_THREADS) {
    const int h = i / dq, j = i - h * dq;
    const T* qs = src + h * (dim + rot);
    if (j < dim) qd[i] = qs[j];
    else if (j >= dimp && j - dimp < rot) qd[i] = from_f32<T>(rotated(qs + dim, j - dimp));
    else qd[i] = from_f32<T>(0.f);
  }
}

template <typename T>
__global__ void ring_gather_kernel(const T* __restrict__ ring, T* __restrict__ latent, const int* __restrict__ slots,
                                   const int* __restrict__ start, int Tn, int P, int ring_len, int lw) {
  const int j = blockIdx.x, b = blockIdx.y;
  const int pos = start[b] - P + j;
  T* dst = latent + ((long long)b * (P + Tn) + j) * lw;
  const bool has = pos >= 0 && pos >= start[b] - ring_len;
  const T* src = ring + ((long long)slots[b] * ring_len + (has ? pos % ring_len : 0)) * lw;
  for (int i = threadIdx.x; i < lw; i += blockDim.x) dst[i] = has ? src[i] : from_f32<T>(0.f);
}

template <typename T>
__global__ void ring_append_kernel(const T* __restrict__ latent, T* __restrict__ ring, const int* __restrict__ slots,
                                   const int* __restrict__ start, const int* __restrict__ count, int Tn, int P, int ring_len, int lw) {
  const int b = blockIdx.y;
  const int t = count[b] - 1 - (int)blockIdx.x;  // newest first
  if (t < 0) return;
  const T* src = latent + ((long long)b * (P + Tn) + P + t) * lw;
  T* dst = ring + ((long long)slots[b] * ring_len + (start[b] + t) % ring_len) * lw;
  for (int i = threadIdx.x; i < lw; i += blockDim.x) dst[i] = src[i];
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
// Per CTA: 16 · MT heads of one sequence against tiles of 64 ring rows. A tile is the key AND the value of all heads, so it is
// fetched once (cp.async, two stages) and read twice from shared memory: S = Q K^T with the rows as the N operand, O += P C
// with the same rows transposed by ldmatrix. N is 64 rows and M 16 or 32 heads, far below a tcgen05 tile, and the
// kernel is bound by the read of the ring.
constexpr int LM_THREADS = 256;
constexpr int LM_KEYS = 64;

__device__ __forceinline__ void lm_cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void lm_ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lm_ldsm2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lm_ldsm2t(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr) : "memory");
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
  int B, heads, dimp, rp, kvp, ring_len, n_split;
  int kv16, ls;            // latent columns rounded up to 16; row pitch in shared memory (elements)
  float scale_log2;
};

// MT: tiles of 16 heads; NTW: tiles of 8 latent columns per warp in the second product
template <int MT, int NTW>
__global__ void __launch_bounds__(LM_THREADS, 1)
latent_decode_mma_kernel(const LmParams p) {
  extern __shared__ __align__(128) uint8_t lm_smem[];
  constexpr int HB = 16 * MT;
  constexpr int SP = LM_KEYS + 1;  // pitch of the score rows
  constexpr int PP = LM_KEYS + 8;  // pitch of the weight rows
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(lm_smem);
  __nv_bfloat16* sk = sq + HB * p.ls;
  __nv_bfloat16* sp = sk + 2 * LM_KEYS * p.ls;
  float* ss = reinterpret_cast<float*>(sp + HB * PP);
  float* sf = ss + HB * SP;  // rescale factor of the tile, per head
  float* sl = sf + HB;       // running sum
  float* smx = sl + HB;      // running maximum
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.x, split = blockIdx.y, h0 = blockIdx.z * HB;
  const int lw = p.kvp + p.rp;
  const int nk = min(p.start[b] + 1, p.ring_len);
  const int nT = (nk + LM_KEYS - 1) / LM_KEYS;
  const int per = (nT + p.n_split - 1) / p.n_split;
  const int ta = split * per, tb = min(nT, ta + per);
  const __nv_bfloat16* base = p.ring + (long long)p.slots[b] * p.ring_len * lw;
  // zero query rows and the padding columns that no copy writes
  {
    const int words = (HB + 2 * LM_KEYS) * p.ls / 8;
    for (int i = tid; i < words; i += LM_THREADS) reinterpret_cast<uint4*>(lm_smem)[i] = make_uint4(0, 0, 0, 0);
    if (tid < HB) {
      sl[tid] = 0.f;
      smx[tid] = -INFINITY;
    }
  }
  __syncthreads();
  const int ku = p.kvp / 8, ru = p.rp / 8, lu = ku + ru;
  auto load_tile = [&](int t, int stage) {
    __nv_bfloat16* dst = sk + stage * LM_KEYS * p.ls;
    const int rows = min(LM_KEYS, nk - t * LM_KEYS);
    for (int i = tid; i < rows * lu; i += LM_THREADS) {
      const int r = i / lu, u = i - r * lu;
      lm_cp_async16(dst + r * p.ls + (u < ku ? u * 8 : p.kv16 + (u - ku) * 8), base + ((long long)(t * LM_KEYS + r)) * lw + u * 8);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (ta < tb) load_tile(ta, 0);
  for (int i = tid; i < HB * lu; i += LM_THREADS) {
    const int h = i / lu, u = i - h * lu;
    if (h0 + h < p.heads) {
      const __nv_bfloat16* src = u < ku ? p.q_abs + ((long long)(h0 + h) * p.B + b) * p.kvp + u * 8
                                        : p.q + ((long long)b * p.heads + h0 + h) * (p.dimp + p.rp) + p.dimp + (u - ku) * 8;
      *reinterpret_cast<uint4*>(sq + h * p.ls + (u < ku ? u * 8 : p.kv16 + (u - ku) * 8)) = *reinterpret_cast<const uint4*>(src);
    }
  }
  float acc[MT][NTW][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NTW; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][j][e] = 0.f;
  const int ksteps = (p.ls - 8) / 16;
  const int n_tiles = p.kv16 / 8;
  // first product: MT = 1: warp -> 8 rows of the tile; MT = 2: warp -> (16 rows, one tile of heads)
  constexpr int NQ = MT == 1 ? 1 : 2;
  const int qm = MT == 1 ? 0 : (warp & 1);
  const int key0 = MT == 1 ? warp * 8 : (warp >> 1) * 16;
  for (int t = ta; t < tb; ++t) {
    const int stage = (t - ta) & 1;
    if (t + 1 < tb) {
      load_tile(t + 1, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const __nv_bfloat16* kt = sk + stage * LM_KEYS * p.ls;
    float s[NQ][4];
#pragma unroll
    for (int i = 0; i < NQ; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
    {
      const uint32_t qa = smem_u32(sq + (qm * 16 + (lane & 15)) * p.ls + (lane >> 4) * 8);
      const uint32_t kb = smem_u32(kt + (key0 + (lane & 7)) * p.ls + ((lane >> 3) & 1) * 8);
#pragma unroll 4
      for (int k = 0; k < ksteps; ++k) {
        uint32_t a[4], b0, b1;
        lm_ldsm4(a, qa + k * 32);
#pragma unroll
        for (int i = 0; i < NQ; ++i) {
          lm_ldsm2(b0, b1, kb + i * 8 * p.ls * 2 + k * 32);
          lm_mma(s[i], a, b0, b1);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int c = key0 + 8 * i + (lane & 3) * 2, r = qm * 16 + (lane >> 2);
      ss[r * SP + c] = s[i][0];
      ss[r * SP + c + 1] = s[i][1];
      ss[(r + 8) * SP + c] = s[i][2];
      ss[(r + 8) * SP + c + 1] = s[i][3];
    }
    __syncthreads();
    const int left = nk - t * LM_KEYS;
#pragma unroll
    for (int i = 0; i < HB / 8; ++i) {
      const int r = warp * (HB / 8) + i;
      const float x0 = lane < left ? ss[r * SP + lane] * p.scale_log2 : -INFINITY;
      const float x1 = lane + 32 < left ? ss[r * SP + lane + 32] * p.scale_log2 : -INFINITY;
      const float mo = smx[r];
      const float mn = fmaxf(mo, warp_max(fmaxf(x0, x1)));
      const float p0 = exp2f(x0 - mn), p1 = exp2f(x1 - mn);
      sp[r * PP + lane] = __float2bfloat16_rn(p0);
      sp[r * PP + lane + 32] = __float2bfloat16_rn(p1);
      const float sum = warp_sum(p0 + p1);
      __syncwarp();
      if (lane == 0) {
        const float f = exp2f(mo - mn);
        sf[r] = f;
        sl[r] = sl[r] * f + sum;
        smx[r] = mn;
      }
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float f0 = sf[m * 16 + (lane >> 2)], f1 = sf[m * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int j = 0; j < NTW; ++j) {
        acc[m][j][0] *= f0;
        acc[m][j][1] *= f0;
        acc[m][j][2] *= f1;
        acc[m][j][3] *= f1;
      }
    }
#pragma unroll
    for (int k = 0; k < LM_KEYS / 16; ++k) {
      uint32_t a[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) lm_ldsm4(a[m], smem_u32(sp + (m * 16 + (lane & 15)) * PP + k * 16 + (lane >> 4) * 8));
      const uint32_t vb = smem_u32(kt + (k * 16 + (lane & 15)) * p.ls);
#pragma unroll
      for (int j = 0; j < NTW; ++j) {
        const int nt = warp * NTW + j;
        if (nt < n_tiles) {
          uint32_t b0, b1;
          lm_ldsm2t(b0, b1, vb + nt * 16);
#pragma unroll
          for (int m = 0; m < MT; ++m) lm_mma(acc[m][j], a[m], b0, b1);
        }
      }
    }
    __syncthreads();  // the stage may be overwritten
  }
  const bool direct = p.n_split == 1;
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = m * 16 + (lane >> 2) + 8 * e, h = h0 + r;
      if (h >= p.heads) continue;
      const float inv = direct ? 1.f / sl[r] : 1.f;
#pragma unroll
      for (int j = 0; j < NTW; ++j) {
        const int c = (warp * NTW + j) * 8 + (lane & 3) * 2;
        if (c >= p.kvp) continue;
        if (direct)
          *reinterpret_cast<uint32_t*>(p.out + ((long long)h * p.B + b) * p.kvp + c) =
              pack_bf16x2(acc[m][j][2 * e] * inv, acc[m][j][2 * e + 1] * inv);
        else
          *reinterpret_cast<float2*>(p.part_o + (((long long)split * p.B + b) * p.heads + h) * p.kvp + c) =
              make_float2(acc[m][j][2 * e], acc[m][j][2 * e + 1]);
      }
    }
  }
  if (!direct && tid < HB && h0 + tid < p.heads) {
    float* ml = p.part_ml + (((long long)split * p.B + b) * p.heads + h0 + tid) * 2;
    ml[0] = smx[tid];
    ml[1] = sl[tid];
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
  long long n = (148 + ctas - 1) / ctas;
  if (n > tiles) n = tiles;
  if (n > 64) n = 64;
  return n < 1 ? 1 : (int)n;
}

static size_t lm_smem_bytes(int mt, int ls) {
  const int hb = 16 * mt;
  return (size_t)(hb + 2 * LM_KEYS) * ls * 2 + (size_t)hb * (LM_KEYS + 8) * 2 + (size_t)hb * (LM_KEYS + 1 + 3) * 4;
}

template <int MT, int NTW>
static int lm_launch(const LmParams& p, cudaStream_t s) {
  const size_t smem = lm_smem_bytes(MT, p.ls);
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(latent_decode_mma_kernel<MT, NTW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
  const dim3 grid(p.B, p.n_split, (p.heads + 16 * MT - 1) / (16 * MT));
  latent_decode_mma_kernel<MT, NTW><<<grid, LM_THREADS, smem, s>>>(p);
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
  KVB_LATENT_TYPES(dtype, (kvb::latent_prep_kernel<T><<<dim3(T_, B), kvb::LP_THREADS, rot_dims * sizeof(float) + 8, (cudaStream_t)stream>>>(
      (const T*)qkv, ld, norm_w, freq, (T*)q, (T*)latent, (T*)ring, slots, start, count, T_, P, ring_len, heads, dim, dimp, rot, rot_dims,
      rp, kv_rank, kvp, eps)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_ring_gather(const void* ring, void* latent, const int* slots, const int* start, int B, int T_, int P, int ring_len,
                               int lw, int dtype, void* stream) {
  if (P <= 0) return KVB_OK;
  if (B <= 0 || B > 65535 || ring_len <= 0) return KVB_ERR_ARG;
  KVB_LATENT_TYPES(dtype, (kvb::ring_gather_kernel<T><<<dim3(P, B), 128, 0, (cudaStream_t)stream>>>((const T*)ring, (T*)latent, slots,
                                                                                                     start, T_, P, ring_len, lw)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

extern "C" int kvb_ring_append(const void* latent, void* ring, const int* slots, const int* start, const int* count, int B, int T_,
                               int P, int ring_len, int lw, int dtype, void* stream) {
  if (B <= 0 || T_ <= 0 || B > 65535 || ring_len <= 0) return KVB_ERR_ARG;
  const int rows = T_ < ring_len ? T_ : ring_len;
  KVB_LATENT_TYPES(dtype, (kvb::ring_append_kernel<T><<<dim3(rows, B), 128, 0, (cudaStream_t)stream>>>((const T*)latent, (T*)ring, slots,
                                                                                                        start, count, T_, P, ring_len, lw)));
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
                                 int simple, void* stream) {
  using namespace kvb;
  if (B <= 0 || heads <= 0 || ring_len <= 0 || B > 65535) return KVB_ERR_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  LmParams p;
  p.kv16 = (kvp + 15) / 16 * 16;
  p.ls = p.kv16 + (rp + 15) / 16 * 16 + 8;
  const int mt = heads > 16 ? 2 : 1;
  if (dtype == 1 && !simple && kvp % 8 == 0 && rp % 8 == 0 && dimp % 8 == 0 && kvp <= 512 && lm_smem_bytes(mt, p.ls) <= 232448) {
    p.q_abs = (const __nv_bfloat16*)q_abs; p.q = (const __nv_bfloat16*)q; p.ring = (const __nv_bfloat16*)ring;
    p.out = (__nv_bfloat16*)out; p.slots = slots; p.start = start;
    p.B = B; p.heads = heads; p.dimp = dimp; p.rp = rp; p.kvp = kvp; p.ring_len = ring_len;
    p.n_split = lm_splits(B, heads, ring_len);
    p.part_o = (float*)scratch;
    p.part_ml = p.part_o + (long long)p.n_split * B * heads * kvp;
    p.scale_log2 = scale * 1.4426950408889634f;
    const int ntw = (p.kv16 / 8 + 7) / 8;
    if (mt == 1) return ntw <= 2 ? lm_launch<1, 2>(p, s) : (ntw <= 4 ? lm_launch<1, 4>(p, s) : lm_launch<1, 8>(p, s));
    return ntw <= 2 ? lm_launch<2, 2>(p, s) : (ntw <= 4 ? lm_launch<2, 4>(p, s) : lm_launch<2, 8>(p, s));
  }
  if (kvp > 32 * LD_MAX_C) return KVB_ERR_TOO_LARGE;
  const size_t smem = ((size_t)kvp + rp + 4 * kvp + 8) * sizeof(float);
  if (smem > 48 * 1024) return KVB_ERR_TOO_LARGE;
  KVB_LATENT_TYPES(dtype, (latent_decode_simple_kernel<T><<<dim3(heads, B), 128, smem, s>>>(
      (const T*)q_abs, (const T*)q, (const T*)ring, (T*)out, slots, start, B, heads, dimp, rp, kvp, ring_len, scale)));
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}
