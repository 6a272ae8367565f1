// Attention of several new tokens on tcgen05, over keys and values expanded from latents, or over the rows of a
// grouped-query cache.
//
//   S = Q_u K_u^T + Q_r K_r^T (the rotated key part K_r is shared by the heads), P = exp2(S·c − m), O += P V
//
// Grouped-query form: no shared part; `group` query heads read one key/value head; keys and values lie in the cache, whose
// rows are the positions of a slot (in a ring, if the layer looks back a bounded way). Optional: one more term in the softmax
// denominator (the running maximum starts at the sink and the sum at 1), soft-capped scores, sigmoid of a gate projection on the output.
// Two maps per head (DIFF): the two query tiles of a CTA are the two maps of the same 128 tokens; they share the value tiles, and the
// epilogue takes the difference of both outputs out of TMEM, norms it per head and stores it.
//
// The head sizes of keys (unrotated + rotated) and values differ and are run-time values: operands are staged as chunks of
// 64 features ([128 rows x 128 B], 128B swizzle, TMA fills what lies beyond a tensor's last feature with zero), S sums over
// the chunks of both parts, and the PV product has N = 64 · (value chunks). One CTA has NQT query tiles of 128 tokens of
// one head, one softmax warpgroup each: with two tiles, one warpgroup works on its scores while the tensor core runs
// PV and the next QK of the other. TMEM: NQT score tiles of 128 columns, NQT outputs of 64 · (value chunks) columns; P
// aliases its S and is the A operand of the PV product.
//
// Masks are arithmetic: key row j of sequence b has position start[b] − P + j (P = start[b] in a grouped-query cache), query t sees
// max(P + t − window + 1, P − start[b], 0) <= j <= P + t. Tiles outside the range of a query tile are skipped, tiles inside
// the range of all its rows need no mask. A grouped query may also see the first `keep` keys, or the means of blocks before its window: their
// tiles come ahead of the others. In a chunked layer its range starts where its chunk does.
#include <cuda.h>
#include <limits.h>

#include <type_traits>

#include "attn_spec.cuh"
#include "common.cuh"
#include "kvb200_layers.h"
#include "tmap.cuh"

namespace kvb {

constexpr int LF_T = 128;
constexpr int LF_CHUNK = LF_T * 128;  // bytes of [128 rows x 64 features]
constexpr int LF_SMEM_LIMIT = 232448;
constexpr int LF_SMEM_MIN = 120 * 1024;  // one CTA per SM: a CTA owns all 512 TMEM columns
constexpr float LF_RESCALE_STEP = 8.f;   // log2 units
constexpr int LF_MAX_STAGES = 4;

struct LfParams {
  __nv_bfloat16* out;
  const int* start;
  int B, heads, T, P, nQ, n_pair;
  int nu, nr, nv;        // feature chunks of the unrotated / rotated key part and of the values
  int ksu_last, ksr;     // 16-feature steps of the last unrotated chunk and of the rotated chunk(s) in total
  int kst, vst;          // stages of K and V
  int vdp, window;
  long long out_ld;
  float scale_log2;
  int* status;
  const int* slots;          // grouped-query cache: slot of every row; NULL: keys and values of the pass
  int group;                 // query heads per key/value head
  const __nv_bfloat16* gate;  // (B, T, gate_ld), or NULL
  long long gate_ld;
  float cap_in, cap_out;      // cap_out > 0: the score in log2 units is cap_out · tanh(cap_in · q·k), and scale_log2 is 1
  kvb_attention a;            // masks, rows, sink, gate columns, difference
};

__device__ __forceinline__ float lf_exp2(float x) { return attn_exp2(x); }

__device__ __forceinline__ void named_barrier(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

__device__ __forceinline__ float lf_sigmoid(float x) { return 1.f / (1.f + __expf(-x)); }

template <int NQT, bool DIFF, bool CAP>
__global__ void __launch_bounds__(64 + 128 * NQT, 1)
latent_flash_kernel(const __grid_constant__ CUtensorMap tmQu, const __grid_constant__ CUtensorMap tmQr,
                    const __grid_constant__ CUtensorMap tmKu, const __grid_constant__ CUtensorMap tmKr,
                    const __grid_constant__ CUtensorMap tmV, const LfParams p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  if (smem_u32(smem) & 1023u) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, STATUS_TIMEOUT_MISC);
    return;
  }
  const int nk = p.nu + p.nr;
  constexpr int MAPS = DIFF ? 2 : 1;  // key tiles of a stage
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + NQT * nk * LF_CHUNK;
  uint8_t* sV = sK + p.kst * MAPS * nk * LF_CHUNK;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + p.vst * p.nv * LF_CHUNK);
  uint64_t* q_full = bars;
  uint64_t* o_full = bars + 1;
  uint64_t* s_full = bars + 2;                 // [NQT]
  uint64_t* p_full = bars + 4;                 // [NQT]
  uint64_t* k_full = bars + 6;                 // [kst]
  uint64_t* k_empty = k_full + LF_MAX_STAGES;
  uint64_t* v_full = k_empty + LF_MAX_STAGES;  // [vst]
  uint64_t* v_empty = v_full + LF_MAX_STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(v_empty + LF_MAX_STAGES);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pair = blockIdx.x % p.n_pair;
  const int h = (blockIdx.x / p.n_pair) % p.heads;
  const int b = blockIdx.x / (p.n_pair * p.heads);
  const int P = p.slots ? p.start[b] : p.P;
  const int lo_seq = max(0, P - p.start[b]);  // first key row that holds a token
  const int hk = h / p.group, bk = p.slots ? p.slots[b] : b;  // where the keys and values are
  auto first_query = [&](int u) { return (DIFF ? pair : pair * NQT + u) * LF_T; };
  // first key that the query at key row hi sees, kept ones aside
  auto seen = [&](int hi) { return max(lo_seq, p.a.chunk > 0 ? hi / p.a.chunk * p.a.chunk : p.window > 0 ? hi - p.window + 1 : 0); };
  // key tiles [ta, tb] of query tile u (empty if the tile has no query)
  auto range = [&](int u, int& ta, int& tb) {
    const int t0 = first_query(u);
    if (t0 >= p.T) {
      ta = INT_MAX;
      tb = -1;
      return;
    }
    const int t1 = min(t0 + LF_T, p.T) - 1;
    ta = seen(P + t0) / LF_T;
    tb = (P + t1) / LF_T;
  };
  int ra[NQT], rb[NQT];
  int first = INT_MAX, last = -1;
#pragma unroll
  for (int u = 0; u < NQT; ++u) {
    range(u, ra[u], rb[u]);
    first = min(first, ra[u]);
    last = max(last, rb[u]);
  }
  // Tiles are counted as they are visited: `kept` ones from the start of the sequence (or of blocks: as many as the last query of the CTA
  // sees), which every query tile visits, then those from `first` on; ra, rb, last are of that count from here on.
  const int keep_tiles = (p.a.keep + LF_T - 1) / LF_T;
  const int last_query = min((DIFF ? pair + 1 : (pair + 1) * NQT) * LF_T, p.T) - 1;
  const int kept = last < 0 ? 0 : p.a.pool ? (blocks_seen(p.a, P + last_query) + LF_T - 1) / LF_T : min(keep_tiles, first), skipped = first - kept;
#pragma unroll
  for (int u = 0; u < NQT; ++u) {
    if (rb[u] < 0) continue;
    if (first < keep_tiles) ra[u] = first;  // some of the kept keys lie behind `first`
    ra[u] -= skipped;
    rb[u] -= skipped;
  }
  if (last >= 0) last -= skipped;
  auto tile_at = [&](int t) { return t < kept ? t : t + skipped; };
  auto visits = [&](int u, int t) { return t >= 0 && t <= rb[u] && (t < kept || t >= ra[u]); };
  auto starts = [&](int u) { return kept > 0 ? 0 : ra[u]; };  // first tile that query tile u visits
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(o_full, 1);
    for (int u = 0; u < NQT; ++u) {
      mbar_init(&s_full[u], 1);
      mbar_init(&p_full[u], 4);
    }
    for (int i = 0; i < LF_MAX_STAGES; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const int o_cols = 64 * p.nv;

  if (warp == 0) {
    // ------------------------------------------------------------ TMA producer
    if (lane == 0) {
      tma_prefetch_desc(&tmQu);
      tma_prefetch_desc(&tmKu);
      if (p.nr > 0) tma_prefetch_desc(&tmQr);
      if (p.nr > 0 || DIFF) tma_prefetch_desc(&tmKr);
      tma_prefetch_desc(&tmV);
      mbar_expect_tx(q_full, (uint32_t)(NQT * nk * LF_CHUNK));
      for (int u = 0; u < NQT; ++u) {
        const int t0 = first_query(u);  // beyond T: zero rows
        for (int c = 0; c < p.nu; ++c) tma_load_4d(sQ + (u * nk + c) * LF_CHUNK, &tmQu, q_full, 64 * c, DIFF ? 2 * h + u : h, t0, b);
        for (int c = 0; c < p.nr; ++c) tma_load_4d(sQ + (u * nk + p.nu + c) * LF_CHUNK, &tmQr, q_full, 64 * c, h, t0, b);
      }
      bool ok = true;
      int ks = 0, vs = 0;
      uint32_t kph = 0, vph = 0;
      for (int t = 0; t <= last; ++t) {
        const int krow = p.a.pool && t < kept ? t * LF_T : p.slots ? row_of(p.a, tile_at(t) * LF_T) : tile_at(t) * LF_T;
        if (!(ok = mbar_wait_bounded(&k_empty[ks], kph ^ 1, abort_flag, p.status, STATUS_TIMEOUT_EMPTY))) break;
        mbar_expect_tx(&k_full[ks], (uint32_t)(MAPS * nk * LF_CHUNK));
        uint8_t* kd = sK + ks * MAPS * nk * LF_CHUNK;
        for (int c = 0; c < p.nu; ++c) tma_load_4d(kd + c * LF_CHUNK, &tmKu, &k_full[ks], 64 * c, hk, krow, bk);
        if (DIFF) {  // keys of the second map
          for (int c = 0; c < p.nu; ++c) tma_load_4d(kd + (p.nu + c) * LF_CHUNK, &tmKr, &k_full[ks], 64 * c, hk, krow, bk);
        } else {
          for (int c = 0; c < p.nr; ++c) tma_load_4d(kd + (p.nu + c) * LF_CHUNK, &tmKr, &k_full[ks], 64 * c, 0, krow, b);
        }
        if (++ks == p.kst) {
          ks = 0;
          kph ^= 1;
        }
        if (!(ok = mbar_wait_bounded(&v_empty[vs], vph ^ 1, abort_flag, p.status, STATUS_TIMEOUT_EMPTY))) break;
        mbar_expect_tx(&v_full[vs], (uint32_t)(p.nv * LF_CHUNK));
        for (int c = 0; c < p.nv; ++c) tma_load_4d(sV + (vs * p.nv + c) * LF_CHUNK, &tmV, &v_full[vs], 64 * c, hk, krow, bk);
        if (++vs == p.vst) {
          vs = 0;
          vph ^= 1;
        }
      }
      if (!ok) {  // copies in flight get a bounded time to land before the shared memory is released
        const long long c0 = clock64();
        while (clock64() - c0 < 2000000LL) {
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(LF_T, LF_T, 0, 0);
      const uint32_t idesc_pv = make_idesc_bf16(LF_T, o_cols, 0, 1);
      const uint32_t q_addr = smem_u32(sQ), k_addr = smem_u32(sK), v_addr = smem_u32(sV);
      const int su = (p.nu - 1) * 4 + p.ksu_last;  // 16-feature steps of the unrotated part
      const int steps = su + p.ksr;
      bool ok = mbar_wait_bounded(q_full, 0, abort_flag, p.status, STATUS_TIMEOUT_FULL);
      int ks = 0, vs = 0;
      uint32_t kph = 0, vph = 0;
      uint32_t pph[NQT];
#pragma unroll
      for (int u = 0; u < NQT; ++u) pph[u] = 0;
      for (int t = 0; t <= last + 1 && ok; ++t) {
        const bool have_k = t <= last, have_v = t > 0;
        bool k_ready = false, v_ready = false;
#pragma unroll
        for (int u = 0; u < NQT; ++u) {
          if (visits(u, t - 1)) {
            if (!v_ready) {
              if (!(ok = mbar_wait_bounded(&v_full[vs], vph, abort_flag, p.status, STATUS_TIMEOUT_FULL))) break;
              v_ready = true;
            }
            if (!(ok = mbar_wait_bounded(&p_full[u], pph[u], abort_flag, p.status, STATUS_TIMEOUT_FULL))) break;
            pph[u] ^= 1;
            tc_fence_after();
#pragma unroll
            for (int kk = 0; kk < 8; ++kk)
              umma_f16_ts(tmem_base + (uint32_t)(NQT * LF_T + u * o_cols), tmem_base + (uint32_t)(u * LF_T + 8 * kk),
                          make_smem_desc_sw128(v_addr + (uint32_t)(vs * p.nv * LF_CHUNK + kk * 16 * 128), LF_CHUNK, 1024), idesc_pv,
                          (t - 1 == starts(u) && kk == 0) ? 0u : 1u);
          }
          if (visits(u, t)) {
            if (!k_ready) {
              if (!(ok = mbar_wait_bounded(&k_full[ks], kph, abort_flag, p.status, STATUS_TIMEOUT_FULL))) break;
              k_ready = true;
            }
            tc_fence_after();
            for (int s = 0; s < steps; ++s) {
              const int c = s < su ? (s >> 2) : p.nu + ((s - su) >> 2);
              const int kk = s < su ? (s & 3) : ((s - su) & 3);
              const uint32_t off = (uint32_t)(c * LF_CHUNK + kk * 32);
              umma_f16_ss(tmem_base + (uint32_t)(u * LF_T), make_smem_desc_sw128(q_addr + (uint32_t)(u * nk * LF_CHUNK) + off, 16, 1024),
                          make_smem_desc_sw128(k_addr + (uint32_t)((ks * MAPS + (DIFF ? u : 0)) * nk * LF_CHUNK) + off, 16, 1024), idesc_qk, s != 0 ? 1u : 0u);
            }
            umma_commit(&s_full[u]);
          }
        }
        if (!ok) break;
        if (have_v) {
          // a tile that no query tile of this CTA visits cannot occur: the ranges overlap or touch
          umma_commit(&v_empty[vs]);
          if (!v_ready && !(ok = mbar_wait_bounded(&v_full[vs], vph, abort_flag, p.status, STATUS_TIMEOUT_FULL))) break;
          if (++vs == p.vst) {
            vs = 0;
            vph ^= 1;
          }
        }
        if (have_k) {
          umma_commit(&k_empty[ks]);
          if (!k_ready && !(ok = mbar_wait_bounded(&k_full[ks], kph, abort_flag, p.status, STATUS_TIMEOUT_FULL))) break;
          if (++ks == p.kst) {
            ks = 0;
            kph ^= 1;
          }
        }
      }
      if (ok) umma_commit(o_full);
    }
  } else {
    // ------------------------------------------------- softmax + epilogue, one warpgroup per query tile
    const int u = NQT == 1 ? 0 : (warp - 2) >> 2;
    const int quarter = warp & 3;
    const int row = quarter * 32 + lane;
    const int t0 = first_query(u);
    const int tq = t0 + row;
    const int my_ra = u == 0 ? ra[0] : ra[NQT - 1], my_rb = u == 0 ? rb[0] : rb[NQT - 1];
    const int my_start = kept > 0 ? 0 : my_ra;
    const int hi = P + tq;
    const int lo = seen(hi);
    // rows of the tile: all see keys in [lo of the last row, hi of the first row] and the kept ones up to the first row
    const int lo_max = seen(P + t0 + LF_T - 1), hi_min = P + t0;
    const int keep = min(p.a.keep, hi + 1);
    const int blocks = blocks_seen(p.a, hi), blocks_min = blocks_seen(p.a, hi_min);  // the fewest of the tile: its first row's
    const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
    const uint32_t tmem_S = tmem_base + (uint32_t)(u * LF_T) + lane_base;
    const uint32_t tmem_O = tmem_base + (uint32_t)(NQT * LF_T + u * o_cols) + lane_base;
    const float c = p.scale_log2;
    const float2 c2 = make_float2(c, c);
    const CapSeries cap(p.cap_in, p.cap_out);
    float m_used = !p.a.sink ? -1e30f : p.a.sink_w ? p.a.sink_w[h] * ATTN_LOG2E : 0.f, l = p.a.sink ? 1.f : 0.f;
    bool ok = true;
    uint32_t ph = 0;
    for (int t = my_start; t <= my_rb; ++t) {
      if (t >= kept && t < my_ra) continue;
      if (!(ok = mbar_wait_bounded(&s_full[u], ph, abort_flag, p.status, STATUS_TIMEOUT_TMEM_FULL))) break;
      ph ^= 1;
      tc_fence_after();
      uint32_t x[LF_T];
#pragma unroll
      for (int w = 0; w < 4; ++w) tmem_ld_32x32b_x32(tmem_S + (uint32_t)(32 * w), x + 32 * w);
      tmem_ld_wait();
      bool series = false;
      if (CAP) {
        // scores well below the cap are capped in the exponent by a series, others (any of the warp's) here by the exponential
        float top = 0.f;
#pragma unroll
        for (int e = 0; e < LF_T; e += 2) top = fmax3(top, fabsf(__uint_as_float(x[e])), fabsf(__uint_as_float(x[e + 1])));
        series = cap.usable() && __all_sync(0xffffffffu, top * p.cap_in <= CAP_SERIES);
        if (!series) {
#pragma unroll
          for (int e = 0; e < LF_T; ++e) x[e] = __float_as_uint(p.cap_out * cap_tanh(__uint_as_float(x[e]) * p.cap_in));
        }
      }
      const int j0 = tile_at(t) * LF_T;
      if (p.a.pool && t < kept) {
        if (j0 + LF_T > blocks_min) {
          const int here = blocks - j0;
#pragma unroll
          for (int e = 0; e < LF_T; ++e)
            if (e >= here) x[e] = 0xff800000u;
        }
      } else if (j0 + LF_T - 1 > hi_min || (j0 < lo_max && j0 + LF_T > p.a.keep)) {
        const uint32_t span = (uint32_t)(hi - lo);
        const uint32_t off = (uint32_t)(j0 - lo);
        const int keep_here = keep - j0;
        if (keep_here <= 0) {
#pragma unroll
          for (int e = 0; e < LF_T; ++e)
            if (off + (uint32_t)e > span) x[e] = 0xff800000u;
        } else {
#pragma unroll
          for (int e = 0; e < LF_T; ++e)
            if (off + (uint32_t)e > span && e >= keep_here) x[e] = 0xff800000u;
        }
      }
      float a8[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) a8[i] = fmaxf(__uint_as_float(x[i]), __uint_as_float(x[8 + i]));
#pragma unroll
      for (int e = 16; e < LF_T; e += 16)
#pragma unroll
        for (int i = 0; i < 8; ++i) a8[i] = fmax3(a8[i], __uint_as_float(x[e + 2 * i]), __uint_as_float(x[e + 2 * i + 1]));
      float m_tile = fmax3(fmax3(a8[0], a8[1], a8[2]), fmax3(a8[3], a8[4], a8[5]), fmaxf(a8[6], a8[7]));
      m_tile = CAP && series ? cap_series(cap, make_float2(m_tile, m_tile), make_float2(0.f, 0.f)).x : m_tile * c;
      const bool raise = m_tile > m_used + LF_RESCALE_STEP;
      const float m_new = raise ? m_tile : m_used;
      // the PV product of the previous tile was issued before this tile's scores: it is complete, O is quiet
      const float f = raise ? lf_exp2(m_used - m_new) : 1.f;
      l *= f;  // at the first tile the sink, if there is one
      if (t > my_start && __any_sync(0xffffffffu, raise)) {
#pragma unroll 1
        for (int c0 = 0; c0 < o_cols; c0 += 16) {
          uint32_t o[16];
          tmem_ld_32x32b_x16(tmem_O + (uint32_t)c0, o);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * f);
          tmem_st_32x32b_x16(tmem_O + (uint32_t)c0, o);
        }
      }
      m_used = m_new;
      const float2 neg_m2 = make_float2(-m_used, -m_used);
      float2 s0 = make_float2(0.f, 0.f), s1 = s0;
      auto weights = [&](auto exponent) {
#pragma unroll
        for (int w = 0; w < 4; ++w) {
          uint32_t pk[16];
#pragma unroll
          for (int e = 0; e < 32; e += 4) {
            const uint32_t* xe = x + 32 * w + e;
            const float2 x0 = exponent(make_float2(__uint_as_float(xe[0]), __uint_as_float(xe[1])));
            const float2 x1 = exponent(make_float2(__uint_as_float(xe[2]), __uint_as_float(xe[3])));
            const float2 y0 = make_float2(lf_exp2(x0.x), lf_exp2(x0.y));
            const float2 y1 = make_float2(lf_exp2(x1.x), lf_exp2(x1.y));
            s0 = fadd2(s0, y0);
            s1 = fadd2(s1, y1);
            pk[e >> 1] = pack_bf16x2(y0.x, y0.y);
            pk[(e >> 1) + 1] = pack_bf16x2(y1.x, y1.y);
          }
          tmem_st_32x32b_x16(tmem_S + (uint32_t)(16 * w), pk);
        }
      };
      if (CAP && series) weights([&](float2 v) { return cap_series(cap, v, neg_m2); });
      else weights([&](float2 v) { return ffma2(v, c2, neg_m2); });
      s0 = fadd2(s0, s1);
      l += s0.x + s0.y;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[u]);
    }
    if (ok) ok = mbar_wait_bounded(o_full, 0, abort_flag, p.status, STATUS_TIMEOUT_TMEM_FULL);
    if (DIFF) {
      // both warpgroups: half of the columns each, of the same rows of both outputs
      __shared__ float s_l[2][LF_T], s_ss[2][LF_T];
      s_l[u][row] = l;
      named_barrier(1, 256);
      tc_fence_after();
      const uint32_t o0 = tmem_base + (uint32_t)(NQT * LF_T) + lane_base, o1 = o0 + (uint32_t)o_cols;
      const float f0 = 1.f / s_l[0][row], f1 = -p.a.lambda / s_l[1][row];
      const int half = o_cols / 2, c_begin = u * half;  // 32 or 64 columns
      float d[64];
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (16 * k >= half) break;
        uint32_t y0[16], y1[16];
        tmem_ld_32x32b_x16(o0 + (uint32_t)(c_begin + 16 * k), y0);
        tmem_ld_32x32b_x16(o1 + (uint32_t)(c_begin + 16 * k), y1);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          d[16 * k + e] = fmaf(__uint_as_float(y1[e]), f1, __uint_as_float(y0[e]) * f0);  // zero in the padding
          ss = fmaf(d[16 * k + e], d[16 * k + e], ss);
        }
      }
      s_ss[u][row] = ss;
      named_barrier(1, 256);
      const float r = p.a.post / sqrtf((s_ss[0][row] + s_ss[1][row]) / (float)p.a.vdim + p.a.eps);
      __nv_bfloat16* dst = p.out + ((long long)b * p.T + (tq < p.T ? tq : 0)) * p.out_ld + h * p.vdp;
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int c = c_begin + 8 * k;
        if (8 * k >= half || c >= p.vdp || tq >= p.T || !ok) break;
        uint4 v;
        v.x = pack_bf16x2(d[8 * k + 0] * r, d[8 * k + 1] * r);
        v.y = pack_bf16x2(d[8 * k + 2] * r, d[8 * k + 3] * r);
        v.z = pack_bf16x2(d[8 * k + 4] * r, d[8 * k + 5] * r);
        v.w = pack_bf16x2(d[8 * k + 6] * r, d[8 * k + 7] * r);
        *reinterpret_cast<uint4*>(dst + c) = v;
      }
    } else if (ok && my_rb >= my_ra) {
      tc_fence_after();
      float inv_l = l > 0.f ? p.a.post / l : 0.f;
      if (p.gate && p.a.gate_cols == 1 && tq < p.T)  // one number per head
        inv_l *= lf_sigmoid(__bfloat162float(p.gate[((long long)b * p.T + tq) * p.gate_ld + h]));
      __nv_bfloat16* dst = p.out + ((long long)b * p.T + (tq < p.T ? tq : 0)) * p.out_ld + h * p.vdp;
#pragma unroll 1
      for (int c0 = 0; c0 < p.vdp; c0 += 16) {
        uint32_t o[16];
        tmem_ld_32x32b_x16(tmem_O + (uint32_t)c0, o);
        tmem_ld_wait();
        if (tq < p.T) {
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            if (c0 + 8 * i >= p.vdp) break;
            if (p.gate && p.a.gate_cols > 1) {
              const uint4 g = *reinterpret_cast<const uint4*>(p.gate + ((long long)b * p.T + tq) * p.gate_ld + h * p.vdp + c0 + 8 * i);
              const uint32_t gw[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[e]));
                o[8 * i + 2 * e] = __float_as_uint(__uint_as_float(o[8 * i + 2 * e]) * lf_sigmoid(f.x));
                o[8 * i + 2 * e + 1] = __float_as_uint(__uint_as_float(o[8 * i + 2 * e + 1]) * lf_sigmoid(f.y));
              }
            }
            uint4 v;
            v.x = pack_bf16x2(__uint_as_float(o[8 * i + 0]) * inv_l, __uint_as_float(o[8 * i + 1]) * inv_l);
            v.y = pack_bf16x2(__uint_as_float(o[8 * i + 2]) * inv_l, __uint_as_float(o[8 * i + 3]) * inv_l);
            v.z = pack_bf16x2(__uint_as_float(o[8 * i + 4]) * inv_l, __uint_as_float(o[8 * i + 5]) * inv_l);
            v.w = pack_bf16x2(__uint_as_float(o[8 * i + 6]) * inv_l, __uint_as_float(o[8 * i + 7]) * inv_l);
            *reinterpret_cast<uint4*>(dst + c0 + 8 * i) = v;
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

struct LfPlan {
  int nqt, nu, nr, nv, kst, vst;
  int smem;
};

// query tiles per CTA and stages that fit into shared and tensor memory; nqt = 0: not supported
static LfPlan lf_plan(int dimp, int rp, int vdp, int maps = 1) {
  LfPlan pl;
  pl.nqt = 0;
  pl.nu = (dimp + 63) / 64;
  pl.nr = (rp + 63) / 64;
  pl.nv = (vdp + 63) / 64;
  const int nk = pl.nu + pl.nr;
  if (dimp <= 0 || rp < 0 || vdp <= 0 || pl.nv > 4) return pl;
  const int limit = LF_SMEM_LIMIT - 512 - (maps == 2 ? 2048 : 0);
  for (int nqt = 2; nqt >= 1; --nqt) {
    if (nqt * (LF_T + 64 * pl.nv) > 512 || nqt < maps) continue;
    static const int stages[][2] = {{3, 3}, {2, 2}, {2, 1}, {1, 2}, {1, 1}};
    for (auto& st : stages) {
      const int bytes = (nqt * nk + st[0] * maps * nk + st[1] * pl.nv) * LF_CHUNK;
      if (bytes > limit || (nqt == 2 && maps == 1 && st[0] == 1)) continue;
      pl.nqt = nqt;
      pl.kst = st[0];
      pl.vst = st[1];
      pl.smem = bytes + 512 < LF_SMEM_MIN ? LF_SMEM_MIN : bytes + 512;
      return pl;
    }
  }
  return pl;
}

template <int NQT, bool DIFF, bool CAP>
static int lf_launch(const CUtensorMap* tm, LfParams& p, int smem, cudaStream_t s) {
  static PerDeviceOnce once;
  if (once.first())
    cudaFuncSetAttribute(latent_flash_kernel<NQT, DIFF, CAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, LF_SMEM_LIMIT - (DIFF ? 2048 : 0));
  p.n_pair = DIFF ? p.nQ : (p.nQ + NQT - 1) / NQT;
  latent_flash_kernel<NQT, DIFF, CAP><<<p.B * p.heads * p.n_pair, 64 + 128 * NQT, smem, s>>>(tm[0], tm[1], tm[2], tm[3], tm[4], p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

}  // namespace kvb

extern "C" int kvb_latent_attend_tc_supported(int dimp, int rp, int vdp) {
  return (dimp % 8 == 0 && rp > 0 && rp % 8 == 0 && vdp % 8 == 0 && kvb::lf_plan(dimp, rp, vdp).nqt > 0) ? 1 : 0;
}

extern "C" int kvb_latent_attend_tc(const void* q, const void* kv, const void* latent, void* out, const int* start, int B, int T, int P,
                                    int heads, int dimp, int rp, int kvp, int vdp, int window, float scale, int* status, void* stream) {
  using namespace kvb;
  if (B <= 0 || T <= 0 || P < 0 || heads <= 0 || window < 0 || !(scale > 0.f)) return KVB_ERR_ARG;
  if ((dimp | rp | vdp | kvp) % 8) return KVB_ERR_ALIGN;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(latent) |
       reinterpret_cast<uintptr_t>(out)) & 15)
    return KVB_ERR_ALIGN;
  const LfPlan pl = lf_plan(dimp, rp, vdp);
  if (!pl.nqt) return KVB_ERR_UNSUPPORTED;
  const uint64_t dq = dimp + rp, row = dimp + vdp, lw = kvp + rp, n = (uint64_t)P + T;
  const uint32_t box[4] = {64, 1, LF_T, 1};
  CUtensorMap tm[5];
  int rc;
  const __nv_bfloat16 *qb = (const __nv_bfloat16*)q, *kb = (const __nv_bfloat16*)kv, *lb = (const __nv_bfloat16*)latent;
  const uint64_t sq[3] = {dq, heads * dq, (uint64_t)T * heads * dq};
  const uint64_t sk[3] = {row, heads * row, n * heads * row};
  const uint64_t sl[3] = {lw, lw, n * lw};
  const uint64_t dqu[4] = {(uint64_t)dimp, (uint64_t)heads, (uint64_t)T, (uint64_t)B}, dqr[4] = {(uint64_t)rp, (uint64_t)heads, (uint64_t)T, (uint64_t)B};
  const uint64_t dku[4] = {(uint64_t)dimp, (uint64_t)heads, n, (uint64_t)B}, dkr[4] = {(uint64_t)rp, 1, n, (uint64_t)B};
  const uint64_t dv[4] = {(uint64_t)vdp, (uint64_t)heads, n, (uint64_t)B};
  if ((rc = tmap_bf16(&tm[0], qb, 4, dqu, sq, box))) return rc;
  if ((rc = tmap_bf16(&tm[1], qb + dimp, 4, dqr, sq, box))) return rc;
  if ((rc = tmap_bf16(&tm[2], kb, 4, dku, sk, box))) return rc;
  if ((rc = tmap_bf16(&tm[3], lb + kvp, 4, dkr, sl, box))) return rc;
  if ((rc = tmap_bf16(&tm[4], kb + dimp, 4, dv, sk, box))) return rc;
  LfParams p;
  p.out = (__nv_bfloat16*)out; p.start = start;
  p.B = B; p.heads = heads; p.T = T; p.P = P; p.nQ = (T + LF_T - 1) / LF_T;
  p.nu = pl.nu; p.nr = pl.nr; p.nv = pl.nv; p.kst = pl.kst; p.vst = pl.vst;
  p.ksu_last = (dimp - 64 * (pl.nu - 1) + 15) / 16;
  p.ksr = (rp + 15) / 16;
  p.vdp = vdp; p.window = window; p.scale_log2 = scale * 1.4426950408889634f; p.status = status;
  p.slots = nullptr; p.group = 1; p.gate = nullptr; p.gate_ld = 0; p.cap_in = p.cap_out = 0.f; p.a = kvb_attention{};
  p.a.post = 1.f; p.out_ld = (long long)heads * vdp;
  return pl.nqt == 2 ? lf_launch<2, false, false>(tm, p, pl.smem, (cudaStream_t)stream) : lf_launch<1, false, false>(tm, p, pl.smem, (cudaStream_t)stream);
}

extern "C" int kvb_grouped_attend_tc_supported(const kvb_attention* a) {
  return (a->dimp % 8 == 0 && a->vdp % 8 == 0 && kvb::lf_plan(a->dimp, 0, a->vdp, a->maps).nqt > 0) ? 1 : 0;
}

extern "C" int kvb_grouped_attend_tc(const void* q, const void* rows, const void* gate, long long gate_ld, void* out, const int* slots,
                                     const int* start, int B, int T, int n_slots, int len, const kvb_attention* a, int* status, void* stream) {
  using namespace kvb;
  if (!a || B <= 0 || T <= 0 || n_slots <= 0 || len <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || !(a->scale > 0.f) ||
      (a->pool && (a->window <= 0 || a->keep || a->ring <= 0)) || a->out_ld < (long long)a->heads * a->vdp || a->out_ld % 8 ||
      (a->maps != 1 && a->maps != 2) || (a->maps == 2 && (a->sink || gate)) || (a->window && a->chunk) || (a->keep && !a->window) ||
      a->head % LF_T || a->ring % LF_T || (a->ring && (a->head < a->keep || a->head + a->ring > len)))
    return KVB_ERR_ARG;
  const int dimp = a->dimp, vdp = a->vdp, maps = a->maps;
  if ((dimp | vdp) % 8 || (gate && a->gate_cols > 1 && (gate_ld % 8 || reinterpret_cast<uintptr_t>(gate) & 15))) return KVB_ERR_ALIGN;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(rows) | reinterpret_cast<uintptr_t>(out)) & 15) return KVB_ERR_ALIGN;
  const LfPlan pl = lf_plan(dimp, 0, vdp, maps);
  if (!pl.nqt) return KVB_ERR_UNSUPPORTED;
  const uint64_t dq = dimp, row = maps * dimp + vdp, H = a->heads * maps, G = a->kv_heads;
  const uint32_t box[4] = {64, 1, LF_T, 1};
  CUtensorMap tm[5];
  int rc;
  const __nv_bfloat16* kb = (const __nv_bfloat16*)rows;
  const uint64_t sq[3] = {dq, H * dq, (uint64_t)T * H * dq};
  const uint64_t sk[3] = {row, G * row, (uint64_t)len * G * row};
  const uint64_t dqu[4] = {dq, H, (uint64_t)T, (uint64_t)B};
  const uint64_t dku[4] = {dq, G, (uint64_t)len, (uint64_t)n_slots}, dv[4] = {(uint64_t)vdp, G, (uint64_t)len, (uint64_t)n_slots};
  if ((rc = tmap_bf16(&tm[0], q, 4, dqu, sq, box))) return rc;
  if ((rc = tmap_bf16(&tm[2], kb, 4, dku, sk, box))) return rc;
  if ((rc = tmap_bf16(&tm[3], kb + (maps - 1) * dimp, 4, dku, sk, box))) return rc;  // one map: never used
  if ((rc = tmap_bf16(&tm[4], kb + maps * dimp, 4, dv, sk, box))) return rc;
  tm[1] = tm[0];  // no shared part: never used
  LfParams p;
  p.out = (__nv_bfloat16*)out; p.start = start;
  p.B = B; p.heads = a->heads; p.T = T; p.P = 0; p.nQ = (T + LF_T - 1) / LF_T;
  p.nu = pl.nu; p.nr = 0; p.nv = pl.nv; p.kst = pl.kst; p.vst = pl.vst;
  p.ksu_last = (dimp - 64 * (pl.nu - 1) + 15) / 16;
  p.ksr = 0;
  p.vdp = vdp; p.window = a->window; p.status = status;
  p.cap_in = a->softcap > 0.f ? a->scale / a->softcap : 0.f;
  p.cap_out = a->softcap * ATTN_LOG2E;
  p.scale_log2 = a->softcap > 0.f ? 1.f : a->scale * ATTN_LOG2E;
  p.slots = slots; p.group = a->heads / a->kv_heads; p.gate = (const __nv_bfloat16*)gate; p.gate_ld = gate_ld; p.a = *a;
  p.out_ld = a->out_ld;
  cudaStream_t s = (cudaStream_t)stream;
  auto launch = [&](auto capped) {
    constexpr bool CAP = decltype(capped)::value;
    if (maps == 2) return lf_launch<2, true, CAP>(tm, p, pl.smem, s);
    return pl.nqt == 2 ? lf_launch<2, false, CAP>(tm, p, pl.smem, s) : lf_launch<1, false, CAP>(tm, p, pl.smem, s);
  };
  return a->softcap > 0.f ? launch(std::true_type{}) : launch(std::false_type{});
}
