// State-space recurrence over several new tokens on tcgen05, in chunks of 128 tokens. With c_t the running sum of the
// logarithms of the decays within a chunk, per head
//
//   y_t = sum_{s <= t} exp(c_t − c_s) dt_s (C_t · B_s) x_s + exp(c_t) S^T C_t + D x_t
//   S'  = exp(c_last) S + sum_s exp(c_last − c_s) dt_s B_s x_s^T
//
// which are four products per chunk: G = C B^T, Y = C S, S += B^T W with W_s = exp(c_last − c_s) dt_s x_s, and Y += P x with P the
// weighted, masked G (D on its diagonal). x, B and C are bf16; everything else is fp32: S stays in TMEM across the chunks of
// a CTA and accumulates there, and P, W and the copy of S that is an operand are each split into a bf16 value and a bf16
// rest, two products instead of one, which keeps 16 bits of their mantissas.
//
// A CTA has one sequence and NH heads of one group, which share the tiles of B and C. One thread feeds tiles (TMA), one warp
// works out step sizes and running sums ahead of the others, one thread per head issues the products, so that the heads drift
// apart and one's products run beside the other's conversions. Two warpgroups per head: both see all rows, each has half of the
// columns. TMEM per head: G (128 columns, P takes its place), Y and S (64 or
// 128 each).
//
// With a fixed decay per head (retention: B the keys, C the queries, x the values) the step size is 1, the running sums are multiples
// of its logarithm and there is no D.
//
// With a decay per token and key channel (gated linear attention, ROWS) queries and keys come with the decays since, and up to, the middle of
// their chunk in them (gated_linear.cu). The state is kept in units of the decay up to that middle: a chunk starts with multiplying its rows
// by (second half of the chunk before) · (first half of this one), which a row of the state is a lane of TMEM for. Nothing else is weighted:
// P is the masked G, and x itself enters the state.
//
// Long passes of few heads are cut into segments: a first launch (STATES) finds what each segment adds to the state and its total
// decay, a small kernel chains them, and the segments then run side by side from their own starting states.
#include <cuda.h>

#include "common.cuh"
#include "kvb200_layers.h"
#include "ssm.cuh"
#include "tmap.cuh"

namespace kvb {

constexpr int SD_T = 128;              // tokens of a chunk
constexpr int SD_TILE = SD_T * 128;    // bytes of [128 rows x 64 columns]
constexpr int SD_SMEM_LIMIT = 232448;
constexpr int SD_FRONT = 128;  // threads of the feeding and issuing warps
constexpr int SD_MAX_SEG = 16;
constexpr float SD_LOG2E = 1.4426950408889634f;

struct SdParams {
  ScanParams s;
  const __nv_bfloat16* u;
  __nv_bfloat16* y;
  float* seg_state;  // (n_seg, B, heads, np, vdp): states at the segments' starts; before the chaining, entry k + 1 holds what k adds
  float* seg_decay;  // (n_seg, B, heads; ROWS: · np): log2 of the segments' decays
  const float* factor;  // ROWS: (B, chunks, heads, np, 2), log2 of the decays of a chunk's halves
  const int* far;       // ROWS: (B, heads), 1: the head is not worked on here
  int chunks;
  int* status;
  int B, n_seg, seg_chunks, n_unit;  // n_unit: CTAs per sequence and segment
};

__device__ __forceinline__ float sd_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void sd_store_4d(const void* tmap, const void* smem, int x, int y, int z, int w) {
  asm volatile("cp.async.bulk.tensor.4d.global.shared::cta.bulk_group [%0, {%2, %3, %4, %5}], [%1];" ::"l"(tmap), "r"(smem_u32(smem)),
               "r"(x), "r"(y), "r"(z), "r"(w) : "memory");
}
// two values as a pair of bf16 (cut off) and the pair of what is missing
__device__ __forceinline__ void sd_split(float2 v, uint32_t& hi, uint32_t& lo) {
  const uint32_t a = __float_as_uint(v.x), b = __float_as_uint(v.y);
  hi = __byte_perm(a, b, 0x7632);
  const float2 r = fadd2(v, make_float2(-__uint_as_float(a & 0xffff0000u), -__uint_as_float(b & 0xffff0000u)));
  lo = pack_bf16x2(r.x, r.y);
}
__device__ __forceinline__ float2 sd_pair(uint32_t a, uint32_t b) { return make_float2(__uint_as_float(a), __uint_as_float(b)); }

template <int NH>
struct SdShared {
  float cum[2][NH][SD_T], dt[2][NH][SD_T];  // of two chunks
  float fac[NH][8][64], total[2][NH];
  uint64_t b_full[2], b_empty[2], c_full, c_empty, d_full[2], d_empty[2];
  uint64_t x_full[NH], x_empty[NH], y_staged[NH], s_ready[NH], g_full[NH], cs_full[NH], w_ready[NH], s_done[NH], p_ready[NH], y_full[NH];
  uint32_t tmem;
  int abort_flag;
};

// NH heads per CTA, NV tiles of 64 value columns, KC tiles of 64 columns of C and B (columns beyond the sizes are zero); STATES: only
// what the segment adds to the state; ROWS: decays by row of the state
template <int NH, int NV, int KC, bool STATES, bool ROWS>
__global__ void __launch_bounds__(SD_FRONT + 256 * NH, 1)
state_scan_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ CUtensorMap tmB, const __grid_constant__ CUtensorMap tmC,
                  const __grid_constant__ CUtensorMap tmY, const SdParams q) {
  extern __shared__ __align__(1024) uint8_t smem[];
  const ScanParams& p = q.s;
  if (smem_u32(smem) & 1023u) {
    if (threadIdx.x == 0 && q.status) atomicCAS(q.status, 0, STATUS_TIMEOUT_MISC);
    return;
  }
  uint8_t* sB = smem;                     // [2 stages][2]: the state product always has 128 rows
  uint8_t* sC = sB + 4 * SD_TILE;         // [KC]
  uint8_t* sX = sC + KC * SD_TILE;        // [NH][NV]: x, then in its place the results on their way out
  uint8_t* sW = sX + NH * NV * SD_TILE;   // [NH][value | rest][NV]: first the state, then W
  SdShared<NH>& sh = *reinterpret_cast<SdShared<NH>*>(sW + 2 * NH * NV * SD_TILE);
  volatile int* abort_flag = &sh.abort_flag;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int unit = blockIdx.x % q.n_unit, seg = blockIdx.x / q.n_unit % q.n_seg, b = blockIdx.x / (q.n_unit * q.n_seg);
  const int h0 = unit * NH, g = h0 / (p.heads / p.groups);
  const int n = p.count[b];
  if (ROWS && q.far[b * p.heads + h0]) return;  // the same for all threads, before anything is set up
  const int ca = seg * q.seg_chunks;
  const int cb = min(ca + q.seg_chunks, (n + SD_T - 1) / SD_T);  // chunks beyond the last real token change nothing
  const int n_chunks = max(0, cb - ca);
  // chunk of turn i. What a segment adds is summed from its end: a chunk's weights then hold the decay up to there, and the sum in
  // TMEM needs no scaling between chunks (ROWS: weights are no number per token, the order is that of time)
  auto chunk_of = [&](int i) { return STATES && !ROWS ? ca + n_chunks - 1 - i : ca + i; };
  constexpr int VC = 64 * NV;
  if (threadIdx.x == 0) {
    mbar_init(&sh.c_full, 1);
    mbar_init(&sh.c_empty, NH);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&sh.b_full[i], 1);
      mbar_init(&sh.b_empty[i], NH);
      mbar_init(&sh.d_full[i], 1);
      mbar_init(&sh.d_empty[i], 8 * NH);
    }
    for (int u = 0; u < NH; ++u) {
      mbar_init(&sh.x_full[u], 1);
      mbar_init(&sh.x_empty[u], ROWS ? 1 : 8);
      mbar_init(&sh.y_staged[u], 8);
      mbar_init(&sh.s_ready[u], 8);
      mbar_init(&sh.g_full[u], 1);
      mbar_init(&sh.cs_full[u], 1);
      mbar_init(&sh.w_ready[u], 8);
      mbar_init(&sh.s_done[u], 1);
      mbar_init(&sh.p_ready[u], 8);
      mbar_init(&sh.y_full[u], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(&sh.tmem, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sh.tmem;
  // TMEM columns of head u: G / P, Y, S
  auto col_g = [&](int u) { return tmem + (uint32_t)(u * (SD_T + 2 * VC)); };
  auto col_y = [&](int u) { return col_g(u) + SD_T; };
  auto col_s = [&](int u) { return col_g(u) + SD_T + VC; };

  if (warp == 0) {
    // ------------------------------------------------------------ TMA producer
    if (lane == 0 && n_chunks > 0) {
      tma_prefetch_desc(&tmX);
      tma_prefetch_desc(&tmB);
      tma_prefetch_desc(&tmC);
      bool ok = true;
      // results of chunk i of head u leave (rows and columns beyond the tensor are cut off); their place is free again afterwards
      auto store = [&](int u, int i) {
        if (!mbar_wait_bounded(&sh.y_staged[u], (uint32_t)(i & 1), abort_flag, q.status, STATUS_TIMEOUT_EMPTY)) return false;
        for (int c = 0; c < NV; ++c) sd_store_4d(&tmY, sX + (u * NV + c) * SD_TILE, 64 * c, h0 + u, (ca + i) * SD_T, b);
        bulk_commit();
        bulk_wait_read_all();
        return true;
      };
      for (int i = 0; i < n_chunks && ok; ++i) {
        const int t0 = chunk_of(i) * SD_T, st = i & 1;
        const uint32_t ph = (uint32_t)(i & 1) ^ 1, bph = (uint32_t)((i >> 1) & 1) ^ 1;
        if (!(ok = mbar_wait_bounded(&sh.b_empty[st], bph, abort_flag, q.status, STATUS_TIMEOUT_EMPTY))) break;
        mbar_expect_tx(&sh.b_full[st], (uint32_t)(2 * SD_TILE));
        for (int c = 0; c < 2; ++c) tma_load_4d(sB + (2 * st + c) * SD_TILE, &tmB, &sh.b_full[st], 64 * c, g, t0, b);  // beyond np: zero
        if (!STATES) {
          if (!(ok = mbar_wait_bounded(&sh.c_empty, ph, abort_flag, q.status, STATUS_TIMEOUT_EMPTY))) break;
          mbar_expect_tx(&sh.c_full, (uint32_t)(KC * SD_TILE));
          for (int c = 0; c < KC; ++c) tma_load_4d(sC + c * SD_TILE, &tmC, &sh.c_full, 64 * c, g, t0, b);
        }
        for (int u = 0; u < NH; ++u) {
          if (STATES) ok = mbar_wait_bounded(&sh.x_empty[u], ph, abort_flag, q.status, STATUS_TIMEOUT_EMPTY);
          else if (i > 0) ok = store(u, i - 1);
          if (!ok) break;
          mbar_expect_tx(&sh.x_full[u], (uint32_t)(NV * SD_TILE));
          for (int c = 0; c < NV; ++c) tma_load_4d(sX + (u * NV + c) * SD_TILE, &tmX, &sh.x_full[u], 64 * c, h0 + u, t0, b);
        }
      }
      if (!STATES) {
        for (int u = 0; u < NH && ok; ++u) ok = store(u, n_chunks - 1);
        bulk_wait_all();
      }
      if (!ok) {  // copies in flight get a bounded time to land before the shared memory is released
        const long long c0 = clock64();
        while (clock64() - c0 < 2000000LL) {
        }
      }
    }
  } else if (warp <= NH) {
    // ------------------------------------------------------------- MMA issuer of head u
    const int u = warp - 1;
    if (lane == 0 && n_chunks > 0) {
      constexpr uint32_t id_g = make_idesc_bf16(SD_T, SD_T, 0, 0);  // C, B both K-major
      constexpr uint32_t id_y = make_idesc_bf16(SD_T, VC, 0, 1);    // A K-major (C) or in TMEM (P), S and x MN-major
      constexpr uint32_t id_s = make_idesc_bf16(SD_T, VC, 1, 1);    // B^T and W MN-major
      // descriptors of the first step of every operand; a step further is an addition to the address field
      constexpr uint64_t STEP_K = 32 >> 4, STEP_MN = (16 * 128) >> 4, TILE = SD_TILE >> 4;
      const uint64_t dC = make_smem_desc_sw128(smem_u32(sC), 16, 1024), dBk = make_smem_desc_sw128(smem_u32(sB), 16, 1024);
      const uint64_t dBt = make_smem_desc_sw128(smem_u32(sB), SD_TILE, 1024);
      const uint64_t dX = make_smem_desc_sw128(smem_u32(sX + u * NV * SD_TILE), SD_TILE, 1024);
      const uint64_t dW = make_smem_desc_sw128(smem_u32(sW + u * 2 * NV * SD_TILE), SD_TILE, 1024);
      const uint32_t tG = col_g(u), tY = col_y(u), tS = col_s(u);
      bool ok = true;
#pragma unroll 1
      for (int i = 0; i < n_chunks && ok; ++i) {
        const uint32_t ph = (uint32_t)(i & 1), bph = (uint32_t)((i >> 1) & 1);
        const int st = i & 1;
        const uint64_t stage = (uint64_t)st * 2 * TILE;
        if (!(ok = mbar_wait_bounded(&sh.b_full[st], bph, abort_flag, q.status, STATUS_TIMEOUT_FULL))) break;
        if (!STATES) {
          if (!(ok = mbar_wait_bounded(&sh.c_full, ph, abort_flag, q.status, STATUS_TIMEOUT_FULL))) break;
        }
        tc_fence_after();
        if (!STATES) {
          // the product with P of the chunk before was issued earlier: G may take its place
#pragma unroll
          for (int k = 0; k < 4 * KC; ++k)
            umma_f16_ss(tG, dC + (k >> 2) * TILE + (k & 3) * STEP_K, dBk + stage + (k >> 2) * TILE + (k & 3) * STEP_K, id_g, k != 0 ? 1u : 0u);
          umma_commit(&sh.g_full[u]);
          if (!(ok = mbar_wait_bounded(&sh.s_ready[u], ph, abort_flag, q.status, STATUS_TIMEOUT_FULL))) break;
          tc_fence_after();
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int k = 0; k < 4 * KC; ++k)
              umma_f16_ss(tY, dC + (k >> 2) * TILE + (k & 3) * STEP_K, dW + part * NV * TILE + k * STEP_MN, id_y, part != 0 || k != 0 ? 1u : 0u);
          if (!ROWS) umma_commit(&sh.cs_full[u]);
          umma_commit(&sh.c_empty);
        }
        if (ROWS) {  // the state has been scaled (s_ready; STATES: w_ready), and x enters as it is
          if (STATES && !(ok = mbar_wait_bounded(&sh.w_ready[u], ph, abort_flag, q.status, STATUS_TIMEOUT_FULL))) break;
          if (!(ok = mbar_wait_bounded(&sh.x_full[u], ph, abort_flag, q.status, STATUS_TIMEOUT_FULL))) break;
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < SD_T / 16; ++k) umma_f16_ss(tS, dBt + stage + k * STEP_MN, dX + k * STEP_MN, id_s, 1u);
          if (STATES) umma_commit(&sh.x_empty[u]);
        } else {
          if (!(ok = mbar_wait_bounded(&sh.w_ready[u], ph, abort_flag, q.status, STATUS_TIMEOUT_FULL))) break;
          tc_fence_after();
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int k = 0; k < SD_T / 16; ++k) umma_f16_ss(tS, dBt + stage + k * STEP_MN, dW + part * NV * TILE + k * STEP_MN, id_s, 1u);
        }
        umma_commit(&sh.s_done[u]);
        umma_commit(&sh.b_empty[st]);
        if (!STATES) {
          if (!ROWS && !(ok = mbar_wait_bounded(&sh.x_full[u], ph, abort_flag, q.status, STATUS_TIMEOUT_FULL))) break;
          if (!(ok = mbar_wait_bounded(&sh.p_ready[u], ph, abort_flag, q.status, STATUS_TIMEOUT_FULL))) break;
          tc_fence_after();
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int k = 0; k < SD_T / 16; ++k) umma_f16_ts(tY, tG + (uint32_t)(32 * (k >> 1) + 16 * part + 8 * (k & 1)), dX + k * STEP_MN, id_y, 1u);
          umma_commit(&sh.y_full[u]);
        }
      }
    }
  } else if (warp == 3) {
    // ------------------- step sizes and running sums (base 2) of the decays, up to two chunks ahead; lane = four tokens.
    // Padding has step 0 and changes nothing. ROWS: nothing to do
    float rate[NH], bias[NH];
#pragma unroll
    for (int u = 0; u < NH && !ROWS; ++u) {
      rate[u] = p.decay ? p.decay[h0 + u] : -expf(p.a_log[h0 + u]) * SD_LOG2E;
      bias[u] = p.decay ? 0.f : p.dt_bias[h0 + u];
    }
    const __nv_bfloat16* raw_dt = p.decay ? nullptr : q.u + (long long)b * p.T * p.ld + p.dt_col + h0;
    float raw[NH][4];
    auto fetch = [&](int i) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = chunk_of(i) * SD_T + 4 * lane + j;
#pragma unroll
        for (int u = 0; u < NH; ++u) raw[u][j] = raw_dt && t < n ? __bfloat162float(raw_dt[(long long)t * p.ld + u]) : 0.f;
      }
    };
    if (n_chunks > 0 && !ROWS) fetch(0);
    bool ok = true;
    for (int i = 0; i < n_chunks && !ROWS; ++i) {
      const int t0 = chunk_of(i) * SD_T + 4 * lane;
      float dt[NH][4], c[NH][4];
#pragma unroll
      for (int u = 0; u < NH; ++u)
#pragma unroll
        for (int j = 0; j < 4; ++j) dt[u][j] = t0 + j >= n ? 0.f : p.decay ? 1.f : ss_softplus_fast(raw[u][j] + bias[u]);
      if (i + 1 < n_chunks) fetch(i + 1);
      if (ok) ok = mbar_wait_bounded(&sh.d_empty[i & 1], (uint32_t)((i >> 1) & 1) ^ 1, abort_flag, q.status, STATUS_TIMEOUT_EMPTY);
#pragma unroll
      for (int u = 0; u < NH; ++u) {
        c[u][0] = rate[u] * dt[u][0];
#pragma unroll
        for (int j = 1; j < 4; ++j) c[u][j] = fmaf(rate[u], dt[u][j], c[u][j - 1]);
        float s = c[u][3];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float v = __shfl_up_sync(0xffffffffu, s, o);
          if (lane >= o) s += v;
        }
        float before = __shfl_up_sync(0xffffffffu, s, 1);
        if (lane == 0) before = 0.f;
        *reinterpret_cast<float4*>(&sh.cum[i & 1][u][4 * lane]) = make_float4(before + c[u][0], before + c[u][1], before + c[u][2], s);
        *reinterpret_cast<float4*>(&sh.dt[i & 1][u][4 * lane]) = make_float4(dt[u][0], dt[u][1], dt[u][2], dt[u][3]);
        if (lane == 31) sh.total[i & 1][u] = s;
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.d_full[i & 1]);
    }
  } else if (warp >= SD_FRONT / 32) {
    // ---------------- head u: thread = row of the tiles (token, or row of the state); warpgroup `half` has half of the columns
    const int u = NH == 1 ? 0 : (warp - SD_FRONT / 32) >> 3, wi = (warp - SD_FRONT / 32) & 7, half = wi >> 2;
    const int quarter = warp & 3, row = quarter * 32 + lane;
    const int h = h0 + u;
    constexpr int HC = VC / 2;  // value columns of a warpgroup
    const int col0 = half * HC;
    const uint32_t lanes = (uint32_t)(quarter * 32) << 16;
    const uint32_t tG = col_g(u) + lanes, tY = col_y(u) + lanes + (uint32_t)col0, tS = col_s(u) + lanes + (uint32_t)col0;
    uint8_t* const w_hi = sW + u * 2 * NV * SD_TILE;
    uint8_t* const w_lo = w_hi + NV * SD_TILE;
    float* const own = p.state + ((long long)p.slots[b] * p.heads + h) * p.np * p.vdp;
    const long long seg_step = (long long)q.B * p.heads * p.np * p.vdp;
    float* const seg_base = q.seg_state ? q.seg_state + ((long long)b * p.heads + h) * p.np * p.vdp : nullptr;
    // starting state of this CTA, NULL: zero
    const float* from = STATES ? nullptr : (q.n_seg > 1 ? seg_base + seg * seg_step : (p.start[b] > 0 ? own : nullptr));
    const float skip = ROWS || p.decay ? 0.f : p.skip[h];
    bool ok = true;  // after a wait that ran out the work goes on unseen: the status word tells, and the loop ends
    float decay_log2 = 0.f;
    auto state_at = [&](const float* base, int c) {  // four columns of this row, zero beyond the sizes
      return row < p.np && col0 + c < p.vdp ? *reinterpret_cast<const float4*>(base + (long long)row * p.vdp + col0 + c)
                                            : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    if (n_chunks > 0) {
#pragma unroll 1
      for (int c0 = 0; c0 < HC; c0 += 16) {
        uint32_t r[16];
#pragma unroll
        for (int e = 0; e < 16; e += 4) {
          const float4 v = from ? state_at(from, c0 + e) : make_float4(0.f, 0.f, 0.f, 0.f);
          r[e] = __float_as_uint(v.x);
          r[e + 1] = __float_as_uint(v.y);
          r[e + 2] = __float_as_uint(v.z);
          r[e + 3] = __float_as_uint(v.w);
        }
        tmem_st_32x32b_x16(tS + (uint32_t)c0, r);
      }
      tmem_st_wait();
    }
    // results of chunk i, once the product with P is there
    auto put_y = [&](int i) {
      if (ok) ok = mbar_wait_bounded(&sh.y_full[u], (uint32_t)(i & 1), abort_flag, q.status, STATUS_TIMEOUT_TMEM_FULL);
      tc_fence_after();
      const bool real = (ca + i) * SD_T + row < n;
#pragma unroll
      for (int c0 = 0; c0 < HC; c0 += 32) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(tY + (uint32_t)c0, r);
        tmem_ld_wait();
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          uint4 v;
          v.x = pack_bf16x2(__uint_as_float(r[8 * k + 0]), __uint_as_float(r[8 * k + 1]));
          v.y = pack_bf16x2(__uint_as_float(r[8 * k + 2]), __uint_as_float(r[8 * k + 3]));
          v.z = pack_bf16x2(__uint_as_float(r[8 * k + 4]), __uint_as_float(r[8 * k + 5]));
          v.w = pack_bf16x2(__uint_as_float(r[8 * k + 6]), __uint_as_float(r[8 * k + 7]));
          const int c = col0 + c0 + 8 * k;
          *reinterpret_cast<uint4*>(sX + (u * NV + c / 64) * SD_TILE + sw128_offset(row, c / 8 & 7)) = real ? v : make_uint4(0u, 0u, 0u, 0u);
        }
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.y_staged[u]);
    };
    // ROWS: log2 of the halves of a chunk's decay of this row
    auto halves = [&](int i) {
      return row < p.np ? *reinterpret_cast<const float2*>(q.factor + ((((long long)b * q.chunks + ca + i) * p.heads + h) * p.np + row) * 2)
                        : make_float2(0.f, 0.f);
    };
    float2 ahead = ROWS && n_chunks > 0 ? halves(0) : make_float2(0.f, 0.f);
    float rest_log2 = 0.f;  // ROWS: second half of the chunk before
#pragma unroll 1
    for (int i = 0; i < n_chunks; ++i) {
      const uint32_t ph = (uint32_t)(i & 1), xph = (uint32_t)((i >> 1) & 1);
      const float* const s_cum = sh.cum[i & 1][u];
      const float* const s_dt = sh.dt[i & 1][u];
      if (!ROWS && ok) ok = mbar_wait_bounded(&sh.d_full[i & 1], xph, abort_flag, q.status, STATUS_TIMEOUT_FULL);
      const float total = ROWS ? ahead.x + ahead.y : sh.total[i & 1][u];
      const float cum = ROWS ? 0.f : s_cum[row], dt = ROWS ? 0.f : s_dt[row];
      const float later = decay_log2;  // STATES: of the chunks behind this one
      decay_log2 += total;
      const float decay = sd_exp2(ROWS ? rest_log2 + ahead.x : total);
      rest_log2 = ahead.y;
      if (ROWS && i + 1 < n_chunks) ahead = halves(i + 1);
      // ---- the state: operand of Y (value and rest), then scaled in place
      if (!STATES && i > 0 && ok) ok = mbar_wait_bounded(&sh.s_done[u], ph ^ 1, abort_flag, q.status, STATUS_TIMEOUT_TMEM_FULL);
      tc_fence_after();
      if (!STATES) {
#pragma unroll
        for (int c0 = 0; c0 < HC; c0 += 32) {
          uint32_t r[32];
          tmem_ld_32x32b_x32(tS + (uint32_t)c0, r);
          tmem_ld_wait();
          const uint32_t tile = (uint32_t)((col0 + c0) / 64 * SD_TILE);
          auto scale = [&]() {
#pragma unroll
            for (int e = 0; e < 32; e += 2) {
              const float2 v = fmul2(sd_pair(r[e], r[e + 1]), make_float2(decay, decay));
              r[e] = __float_as_uint(v.x);
              r[e + 1] = __float_as_uint(v.y);
            }
          };
          if (ROWS) scale();  // queries meet the state in the same units
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) sd_split(sd_pair(r[8 * k + 2 * e], r[8 * k + 2 * e + 1]), hi[e], lo[e]);
            const uint32_t off = tile + sw128_offset(row, ((col0 + c0) & 63) / 8 + k);
            *reinterpret_cast<uint4*>(w_hi + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(w_lo + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
          if (!ROWS) scale();
          tmem_st_32x32b_x16(tS + (uint32_t)c0, r);
          tmem_st_32x32b_x16(tS + (uint32_t)(c0 + 16), r + 16);
        }
        tmem_st_wait();
        fence_proxy_async_smem();
        if (i > 0) put_y(i - 1);  // before the next Y takes its place
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&sh.s_ready[u]);
        // ---- P, blocks of 32 tokens: the first warpgroup has blocks 0 and 3, the second 1 and 2. In blocks before this warp's rows the
        // factor is one of the row times one of the column, both at most 1
        if (ok) ok = mbar_wait_bounded(&sh.g_full[u], ph, abort_flag, q.status, STATUS_TIMEOUT_TMEM_FULL);
        tc_fence_after();
        const float ref = !ROWS && quarter > 0 ? s_cum[32 * quarter - 1] : 0.f;
        const float rf = sd_exp2(cum - ref);
        const float2 rf2 = make_float2(rf, rf);
        float* const fac = sh.fac[u][wi];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int k = j == 0 ? half : 3 - half;
          if (!ROWS && k < quarter) fac[32 * j + lane] = sd_exp2(ref - s_cum[32 * k + lane]) * s_dt[32 * k + lane];
        }
        __syncwarp();
#pragma unroll 1
        for (int j = 0; j < 2; ++j) {
          const int k = j == 0 ? half : 3 - half;
          uint32_t x[32];
          if (k <= quarter) {
            tmem_ld_32x32b_x32(tG + (uint32_t)(32 * k), x);
            tmem_ld_wait();
          }
          uint32_t hi[16], lo[16];
          if (ROWS && k <= quarter) {
            // behind the diagonal keys are not weighted down: what they give there may be anything
#pragma unroll
            for (int e = 0; e < 32; e += 2) {
              if (k == quarter && e > lane) x[e] = 0u;
              if (k == quarter && e + 1 > lane) x[e + 1] = 0u;
              sd_split(sd_pair(x[e], x[e + 1]), hi[e / 2], lo[e / 2]);
            }
          } else if (k < quarter) {
#pragma unroll
            for (int e = 0; e < 32; e += 4) {
              const float4 f = *reinterpret_cast<const float4*>(fac + 32 * j + e);
              const uint32_t* xe = x + e;
              sd_split(fmul2(sd_pair(xe[0], xe[1]), fmul2(rf2, make_float2(f.x, f.y))), hi[e / 2], lo[e / 2]);
              sd_split(fmul2(sd_pair(xe[2], xe[3]), fmul2(rf2, make_float2(f.z, f.w))), hi[e / 2 + 1], lo[e / 2 + 1]);
            }
          } else if (k == quarter) {
#pragma unroll
            for (int e = 0; e < 32; e += 4) {
              const float4 cs = *reinterpret_cast<const float4*>(s_cum + 32 * k + e), ds = *reinterpret_cast<const float4*>(s_dt + 32 * k + e);
              const float cc[4] = {cs.x, cs.y, cs.z, cs.w}, dd[4] = {ds.x, ds.y, ds.z, ds.w};
              float v[4];
#pragma unroll
              for (int c = 0; c < 4; ++c) {
                v[c] = __uint_as_float(x[e + c]) * (sd_exp2(cum - cc[c]) * dd[c]);
                if (e + c > lane) v[c] = 0.f;
                if (e + c == lane) v[c] += skip;
              }
              sd_split(make_float2(v[0], v[1]), hi[e / 2], lo[e / 2]);
              sd_split(make_float2(v[2], v[3]), hi[e / 2 + 1], lo[e / 2 + 1]);
            }
          } else {
#pragma unroll
            for (int e = 0; e < 16; ++e) hi[e] = lo[e] = 0u;
          }
          // in the place of the columns it was made of: values, then rests
          tmem_st_32x32b_x16(tG + (uint32_t)(32 * k), hi);
          tmem_st_32x32b_x16(tG + (uint32_t)(32 * k + 16), lo);
        }
      }
      if constexpr (ROWS) {
        if (STATES) {
          if (i > 0) {  // at first the state is zero
            if (ok) ok = mbar_wait_bounded(&sh.s_done[u], ph ^ 1, abort_flag, q.status, STATUS_TIMEOUT_TMEM_FULL);
            tc_fence_after();
#pragma unroll
            for (int c0 = 0; c0 < HC; c0 += 32) {
              uint32_t r[32];
              tmem_ld_32x32b_x32(tS + (uint32_t)c0, r);
              tmem_ld_wait();
#pragma unroll
              for (int e = 0; e < 32; e += 2) {
                const float2 v = fmul2(sd_pair(r[e], r[e + 1]), make_float2(decay, decay));
                r[e] = __float_as_uint(v.x);
                r[e + 1] = __float_as_uint(v.y);
              }
              tmem_st_32x32b_x16(tS + (uint32_t)c0, r);
              tmem_st_32x32b_x16(tS + (uint32_t)(c0 + 16), r + 16);
            }
          }
        }
        tmem_st_wait();  // the scaled state, or P
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(STATES ? &sh.w_ready[u] : &sh.p_ready[u]);
        continue;
      }
      // ---- W, in the place of the state's copy once that has been used
      if (ok) ok = mbar_wait_bounded(&sh.x_full[u], ph, abort_flag, q.status, STATUS_TIMEOUT_FULL);
      const uint8_t* xt = sX + u * NV * SD_TILE;
      const float wf = sd_exp2(STATES ? later + (total - cum) : total - cum) * dt;
      uint4 xv[HC / 8];
#pragma unroll
      for (int k = 0; k < HC / 8; ++k)
        xv[k] = *reinterpret_cast<const uint4*>(xt + (col0 + 8 * k) / 64 * SD_TILE + sw128_offset(row, ((col0 & 63) / 8 + k) & 7));
      if (STATES) {
        __syncwarp();
        if (lane == 0) mbar_arrive(&sh.x_empty[u]);
        if (i > 0 && ok) ok = mbar_wait_bounded(&sh.s_done[u], ph ^ 1, abort_flag, q.status, STATUS_TIMEOUT_TMEM_FULL);
      } else if (ok) {
        ok = mbar_wait_bounded(&sh.cs_full[u], ph, abort_flag, q.status, STATUS_TIMEOUT_TMEM_FULL);
      }
#pragma unroll
      for (int k = 0; k < HC / 8; ++k) {
        const uint32_t off = (uint32_t)((col0 + 8 * k) / 64 * SD_TILE) + sw128_offset(row, ((col0 & 63) / 8 + k) & 7);
        const uint32_t xw[4] = {xv[k].x, xv[k].y, xv[k].z, xv[k].w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) sd_split(fmul2(sd_pair(xw[e] << 16, xw[e] & 0xffff0000u), make_float2(wf, wf)), hi[e], lo[e]);
        *reinterpret_cast<uint4*>(w_hi + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(w_lo + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(&sh.w_ready[u]);
        mbar_arrive(&sh.d_empty[i & 1]);
      }
      if (STATES) continue;
      // ---- Y so far is C S: the decay since the chunk's start
      tc_fence_after();
      const float since = sd_exp2(cum);
#pragma unroll
      for (int c0 = 0; c0 < HC; c0 += 32) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(tY + (uint32_t)c0, r);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e += 2) {
          const float2 v = fmul2(sd_pair(r[e], r[e + 1]), make_float2(since, since));
          r[e] = __float_as_uint(v.x);
          r[e + 1] = __float_as_uint(v.y);
        }
        tmem_st_32x32b_x16(tY + (uint32_t)c0, r);
        tmem_st_32x32b_x16(tY + (uint32_t)(c0 + 16), r + 16);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.p_ready[u]);
    }
    if (!STATES && n_chunks > 0) put_y(n_chunks - 1);
    // ---- what is left of the segment is padding
    if (!STATES) {
      for (int t = (ca + n_chunks) * SD_T + row; t < min((ca + q.seg_chunks) * SD_T, p.T); t += SD_T)
        for (int c0 = col0; c0 < min(col0 + HC, p.vdp); c0 += 8)
          *reinterpret_cast<uint4*>(q.y + ((long long)b * p.T + t) * p.inner + h * p.vdp + c0) = make_uint4(0u, 0u, 0u, 0u);
    }
    // ---- the state goes on: to the chaining kernel, or (last segment) to its sequence
    if (n_chunks > 0 && ok) ok = mbar_wait_bounded(&sh.s_done[u], (uint32_t)((n_chunks - 1) & 1), abort_flag, q.status, STATUS_TIMEOUT_TMEM_FULL);
    tc_fence_after();
    const float last = ROWS ? sd_exp2(rest_log2) : 1.f;  // to the end of the last chunk
    float* const to = STATES ? seg_base + (seg + 1) * seg_step : (seg == q.n_seg - 1 && n > 0 ? own : nullptr);
    if (to && ok) {
#pragma unroll 1
      for (int c0 = 0; c0 < HC; c0 += 16) {
        uint32_t r[16];
        if (n_chunks > 0) {
          tmem_ld_32x32b_x16(tS + (uint32_t)c0, r);
          tmem_ld_wait();
        }
#pragma unroll
        for (int e = 0; e < 16; e += 4) {
          float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
          if (n_chunks > 0)
            v = make_float4(__uint_as_float(r[e]) * last, __uint_as_float(r[e + 1]) * last, __uint_as_float(r[e + 2]) * last, __uint_as_float(r[e + 3]) * last);
          else if (from)
            v = state_at(from, c0 + e);
          if (row < p.np && col0 + c0 + e < p.vdp) *reinterpret_cast<float4*>(to + (long long)row * p.vdp + col0 + c0 + e) = v;
        }
      }
    }
    if (ROWS) {
      if (STATES && half == 0 && row < p.np) q.seg_decay[(((long long)(seg + 1) * q.B + b) * p.heads + h) * p.np + row] = decay_log2;
    } else if (STATES && row == 0 && half == 0) q.seg_decay[((long long)(seg + 1) * q.B + b) * p.heads + h] = decay_log2;
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// Starting states of the segments: entry 0 is the sequence's state, entry k + 1 what segment k makes of entry k.
constexpr int SD_CHAIN = 256;

template <bool ROWS>
__global__ void __launch_bounds__(SD_CHAIN)
state_chain_kernel(const SdParams q) {
  const ScanParams& p = q.s;
  const int h = blockIdx.y, b = blockIdx.z, i = blockIdx.x * SD_CHAIN + threadIdx.x;
  const long long size = (long long)p.np * p.vdp, step = (long long)q.B * p.heads * size / 4;
  if (i >= size / 4 || (ROWS && q.far[b * p.heads + h])) return;
  const int row = ROWS ? 4 * i / p.vdp : 0, rows = ROWS ? p.np : 1;  // of the decays
  const float4* own = reinterpret_cast<const float4*>(p.state + ((long long)p.slots[b] * p.heads + h) * size);
  float4* seg = reinterpret_cast<float4*>(q.seg_state + ((long long)b * p.heads + h) * size) + i;
  float4 s = p.start[b] > 0 ? own[i] : make_float4(0.f, 0.f, 0.f, 0.f);
  seg[0] = s;
#pragma unroll 4
  for (int k = 1; k < q.n_seg; ++k) {
    const float f = sd_exp2(q.seg_decay[(((long long)k * q.B + b) * p.heads + h) * rows + row]);
    const float4 add = seg[k * step];
    s = make_float4(fmaf(f, s.x, add.x), fmaf(f, s.y, add.y), fmaf(f, s.z, add.z), fmaf(f, s.w, add.w));
    seg[k * step] = s;
  }
}

struct SdPlan {
  int nh, nv, kc, n_seg, seg_chunks, smem;
};

static SdPlan sd_plan(int B, int T, int heads, int groups, int vdp, int np) {
  SdPlan pl;
  pl.nv = (vdp + 63) / 64;
  pl.nh = pl.nv == 1 && heads / groups % 2 == 0 ? 2 : 1;
  pl.kc = (np + 63) / 64;
  const int tiles = 4 + pl.kc + 3 * pl.nh * pl.nv;
  pl.smem = tiles * SD_TILE + (int)(pl.nh == 2 ? sizeof(SdShared<2>) : sizeof(SdShared<1>));
  if (pl.smem < 120 * 1024) pl.smem = 120 * 1024;  // one CTA per SM: a CTA owns all 512 TMEM columns
  const int chunks = (T + SD_T - 1) / SD_T;
  const long long ctas = (long long)B * heads / pl.nh;
  long long n = 148 / ctas;
  if (n > chunks / 4) n = chunks / 4;
  if (n > SD_MAX_SEG) n = SD_MAX_SEG;
  if (n < 2) n = 1;
  pl.seg_chunks = (int)((chunks + n - 1) / n);
  pl.n_seg = (chunks + pl.seg_chunks - 1) / pl.seg_chunks;
  return pl;
}

template <int NH, int NV, int KC, bool ROWS>
static int sd_launch(const CUtensorMap* tm, SdParams& q, int smem, cudaStream_t s) {
  static PerDeviceOnce once;
  if (once.first()) {
    cudaFuncSetAttribute(state_scan_kernel<NH, NV, KC, false, ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, SD_SMEM_LIMIT);
    cudaFuncSetAttribute(state_scan_kernel<NH, NV, KC, true, ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, SD_SMEM_LIMIT);
  }
  q.n_unit = q.s.heads / NH;
  const int per_seg = q.n_unit * q.B, n_seg = q.n_seg;
  if (n_seg > 1) {
    q.n_seg = n_seg - 1;  // what the last segment adds is nobody's start
    state_scan_kernel<NH, NV, KC, true, ROWS><<<per_seg * (n_seg - 1), SD_FRONT + 256 * NH, smem, s>>>(tm[0], tm[1], tm[2], tm[3], q);
    q.n_seg = n_seg;
    state_chain_kernel<ROWS><<<dim3((q.s.np * q.s.vdp / 4 + SD_CHAIN - 1) / SD_CHAIN, q.s.heads, q.B), SD_CHAIN, 0, s>>>(q);
  }
  state_scan_kernel<NH, NV, KC, false, ROWS><<<per_seg * n_seg, SD_FRONT + 256 * NH, smem, s>>>(tm[0], tm[1], tm[2], tm[3], q);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

}  // namespace kvb

extern "C" int kvb_state_scan_tc_supported(int heads, int groups, int vdp, int np) {
  return heads > 0 && groups > 0 && heads % groups == 0 && vdp % 8 == 0 && np % 8 == 0 && vdp > 0 && np > 0 && vdp <= 128 && np <= 128;
}

extern "C" long long kvb_state_scan_tc_scratch_bytes(int B, int T, int heads, int groups, int vdp, int np) {
  const kvb::SdPlan pl = kvb::sd_plan(B, T, heads, groups, vdp, np);
  return pl.n_seg > 1 ? (long long)pl.n_seg * B * heads * ((long long)np * vdp + 1) * 4 : 0;
}

namespace kvb {

// What both recurrences hand over: values x (ldx), keys B and queries C (ldb) of every token, heads in groups that share B and C.
static int sd_run(SdParams& q, const __nv_bfloat16* x, long long ldx, const __nv_bfloat16* bm, const __nv_bfloat16* cm, long long ldb,
                  float* scratch, cudaStream_t s) {
  const ScanParams& p = q.s;
  const int B = q.B, T = p.T;
  if (B <= 0 || B > 65535 || T <= 0) return KVB_ERR_ARG;
  if (!kvb_state_scan_tc_supported(p.heads, p.groups, p.vdp, p.np)) return KVB_ERR_UNSUPPORTED;
  if ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(bm) | reinterpret_cast<uintptr_t>(cm) | reinterpret_cast<uintptr_t>(q.y) |
       reinterpret_cast<uintptr_t>(p.state) | reinterpret_cast<uintptr_t>(scratch)) & 15 || ldx % 8 || ldb % 8)
    return KVB_ERR_ALIGN;
  const SdPlan pl = sd_plan(B, T, p.heads, p.groups, p.vdp, p.np);
  if (pl.smem > SD_SMEM_LIMIT) return KVB_ERR_TOO_LARGE;
  if (pl.n_seg > 1 && !scratch) return KVB_ERR_ARG;
  q.n_seg = pl.n_seg;
  q.seg_chunks = pl.seg_chunks;
  q.seg_state = pl.n_seg > 1 ? scratch : nullptr;
  q.seg_decay = pl.n_seg > 1 ? scratch + (long long)pl.n_seg * B * p.heads * p.np * p.vdp : nullptr;
  const uint32_t box[4] = {64, 1, SD_T, 1};
  CUtensorMap tm[4];
  int rc;
  const uint64_t lx = ldx, lb = ldb;
  const uint64_t dx[4] = {(uint64_t)p.vdp, (uint64_t)p.heads, (uint64_t)T, (uint64_t)B}, sx[3] = {(uint64_t)p.vdp, lx, T * lx};
  const uint64_t db[4] = {(uint64_t)p.np, (uint64_t)p.groups, (uint64_t)T, (uint64_t)B}, sb[3] = {(uint64_t)p.np, lb, T * lb};
  if ((rc = tmap_bf16(&tm[0], x, 4, dx, sx, box))) return rc;
  if ((rc = tmap_bf16(&tm[1], bm, 4, db, sb, box))) return rc;
  if ((rc = tmap_bf16(&tm[2], cm, 4, db, sb, box))) return rc;
  const uint64_t sy[3] = {(uint64_t)p.vdp, (uint64_t)p.inner, (uint64_t)T * p.inner};
  if ((rc = tmap_bf16(&tm[3], q.y, 4, dx, sy, box))) return rc;
  if (q.factor) {  // heads do not share keys
    if (pl.nv == 1) return pl.kc == 1 ? sd_launch<1, 1, 1, true>(tm, q, pl.smem, s) : sd_launch<1, 1, 2, true>(tm, q, pl.smem, s);
    return pl.kc == 1 ? sd_launch<1, 2, 1, true>(tm, q, pl.smem, s) : sd_launch<1, 2, 2, true>(tm, q, pl.smem, s);
  }
  if (pl.nh == 2) return pl.kc == 1 ? sd_launch<2, 1, 1, false>(tm, q, pl.smem, s) : sd_launch<2, 1, 2, false>(tm, q, pl.smem, s);
  if (pl.nv == 1) return pl.kc == 1 ? sd_launch<1, 1, 1, false>(tm, q, pl.smem, s) : sd_launch<1, 1, 2, false>(tm, q, pl.smem, s);
  return pl.kc == 1 ? sd_launch<1, 2, 1, false>(tm, q, pl.smem, s) : sd_launch<1, 2, 2, false>(tm, q, pl.smem, s);
}

}  // namespace kvb

extern "C" int kvb_state_scan_tc(const void* u, long long ld, int dt_col, const void* xbc, const float* dt_bias, const float* a_log,
                                 const float* skip, float* state, void* y, void* scratch, const int* slots, const int* start,
                                 const int* count, int B, int T, int heads, int groups, int vdp, int np, int* status, void* stream) {
  using namespace kvb;
  SdParams q;
  ScanParams& p = q.s;
  p.dt_bias = dt_bias; p.a_log = a_log; p.skip = skip; p.decay = nullptr; p.slots = slots; p.start = start; p.count = count;
  p.state = state; p.ld = ld; p.T = T; p.dt_col = dt_col; p.heads = heads; p.groups = groups; p.vdp = vdp; p.np = np; p.inner = heads * vdp;
  p.channels = heads * vdp + 2 * groups * np;
  q.u = (const __nv_bfloat16*)u; q.y = (__nv_bfloat16*)y; q.status = status; q.B = B;
  q.factor = nullptr; q.far = nullptr; q.chunks = 0;
  const __nv_bfloat16* x = (const __nv_bfloat16*)xbc;
  return sd_run(q, x, p.channels, x + p.inner, x + p.inner + groups * np, p.channels, (float*)scratch, (cudaStream_t)stream);
}

extern "C" int kvb_retention_scan_tc(const void* v, long long ldv, const void* qk, long long ldqk, const float* log2_decay, float* state,
                                     void* y, void* scratch, const int* slots, const int* start, const int* count, int B, int T, int heads,
                                     int vdp, int np, int* status, void* stream) {
  using namespace kvb;
  if (!log2_decay) return KVB_ERR_ARG;
  SdParams q;
  ScanParams& p = q.s;
  p.dt_bias = p.a_log = p.skip = nullptr; p.decay = log2_decay; p.slots = slots; p.start = start; p.count = count; p.state = state;
  p.ld = 0; p.T = T; p.dt_col = 0; p.heads = heads; p.groups = heads; p.vdp = vdp; p.np = np; p.inner = heads * vdp; p.channels = 0;
  q.u = nullptr; q.y = (__nv_bfloat16*)y; q.status = status; q.B = B;
  q.factor = nullptr; q.far = nullptr; q.chunks = 0;
  const __nv_bfloat16* c = (const __nv_bfloat16*)qk;
  return sd_run(q, (const __nv_bfloat16*)v, ldv, c + heads * np, c, ldqk, (float*)scratch, (cudaStream_t)stream);
}

extern "C" long long kvb_gated_linear_scan_tc_scratch_bytes(int B, int T, int heads, int vdp, int np) {
  const kvb::SdPlan pl = kvb::sd_plan(B, T, heads, heads, vdp, np);
  return pl.n_seg > 1 ? (long long)pl.n_seg * B * heads * np * ((long long)vdp + 1) * 4 : 0;
}

extern "C" int kvb_gated_linear_scan_tc(const void* v, long long ldv, const void* qk, const float* factor, const int* far, float* state, void* y,
                                        void* scratch, const int* slots, const int* start, const int* count, int B, int T, int heads, int vdp,
                                        int np, int* status, void* stream) {
  using namespace kvb;
  if (!factor || !far) return KVB_ERR_ARG;
  SdParams q;
  ScanParams& p = q.s;
  p.dt_bias = p.a_log = p.skip = p.decay = nullptr; p.slots = slots; p.start = start; p.count = count; p.state = state;
  p.ld = 0; p.T = T; p.dt_col = 0; p.heads = heads; p.groups = heads; p.vdp = vdp; p.np = np; p.inner = heads * vdp; p.channels = 0;
  q.u = nullptr; q.y = (__nv_bfloat16*)y; q.status = status; q.B = B;
  q.factor = factor; q.far = far; q.chunks = (T + SD_T - 1) / SD_T;
  const __nv_bfloat16* c = (const __nv_bfloat16*)qk;
  return sd_run(q, (const __nv_bfloat16*)v, ldv, c + heads * np, c, 2 * heads * np, (float*)scratch, (cudaStream_t)stream);
}
