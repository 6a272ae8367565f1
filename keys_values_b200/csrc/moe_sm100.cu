// Grouped bf16 product of routed experts on tcgen05:  out[r, :] = act(W_e · in[r, :]) for rows sorted by expert.
//
// The expert's weight rows are the M = 128 operand and the tokens the N operand, so a tile is 128 features x `tile`
// tokens with tile = 16 .. 256 chosen by the caller from the expected number of tokens per expert: prefill takes wide
// tiles, a decode step with a few tokens per expert streams each weight once without padding the tokens to 128 rows.
// Persistent CTAs over a device-side tile table (token tile, expert), the structure of the plain GEMM of this package:
// warp 0 TMA producer (ring of 128B-swizzled stages), warp 1 MMA issuer with a double-buffered accumulator in TMEM,
// warps 2..5 epilogue (activation, bf16, stores of two tokens per instruction). In a gated unit (act 2) weight rows 2 f and 2 f + 1 are
// gate and up projection of result f: neighbouring lanes exchange what the other needs and each has silu(gate) · up of every other token.
#include <cuda.h>

#include "common.cuh"
#include "kvb200_layers.h"
#include "tmap.cuh"

namespace kvb {

constexpr int MG_M = 128, MG_K = 64, MG_THREADS = 192, MG_MAX_STAGES = 8;
constexpr int MG_A_BYTES = MG_M * MG_K * 2;
constexpr int MG_SMEM_LIMIT = 224 * 1024;

struct MgParams {
  __nv_bfloat16* out;
  const int *plan, *tile_expert, *tile_row;
  int tile, n_out, k, stages, act;
  long long ldo;
  int* status;
};

__global__ void __launch_bounds__(MG_THREADS, 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmX, const MgParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int stage_bytes = MG_A_BYTES + p.tile * MG_K * 2;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + p.stages * stage_bytes);
  uint64_t* empty_bar = full_bar + MG_MAX_STAGES;
  uint64_t* tmem_full = empty_bar + MG_MAX_STAGES;
  uint64_t* tmem_empty = tmem_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tmem_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int num_f = (p.n_out + MG_M - 1) / MG_M;
  const int num_tiles = p.plan[0] * num_f;
  const int num_kb = (p.k + MG_K - 1) / MG_K;
  const int tmem_cols = 2 * p.tile < 32 ? 32 : 2 * p.tile;

  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(&tmem_full[a], 1);
      mbar_init(&tmem_empty[a], 4);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      tma_prefetch_desc(&tmW);
      tma_prefetch_desc(&tmX);
      int stage = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
        const int ti = tile / num_f, f0 = (tile % num_f) * MG_M;
        const int wrow = p.tile_expert[ti] * p.n_out + f0, xrow = p.tile_row[ti];
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!(ok = mbar_wait_bounded(&empty_bar[stage], phase ^ 1, abort_flag, p.status, STATUS_TIMEOUT_EMPTY))) break;
          uint8_t* sa = smem + stage * stage_bytes;
          mbar_expect_tx(&full_bar[stage], (uint32_t)stage_bytes);
          tma_load_2d(sa, &tmW, &full_bar[stage], kb * MG_K, wrow);
          tma_load_2d(sa + MG_A_BYTES, &tmX, &full_bar[stage], kb * MG_K, xrow);
          if (++stage == p.stages) {
            stage = 0;
            phase ^= 1;
          }
        }
      }
      if (!ok) {  // copies in flight get a bounded time to land before the shared memory is released
        const long long c0 = clock64();
        while (clock64() - c0 < 2000000LL) {
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = make_idesc_bf16(MG_M, p.tile, 0, 0);
      int stage = 0, acc = 0;
      uint32_t phase = 0, acc_phase = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
        if (!mbar_wait_bounded(&tmem_empty[acc], acc_phase ^ 1, abort_flag, p.status, STATUS_TIMEOUT_TMEM_EMPTY)) break;
        tc_fence_after();
        const uint32_t d_tmem = tmem_base + (uint32_t)(acc * p.tile);
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!(ok = mbar_wait_bounded(&full_bar[stage], phase, abort_flag, p.status, STATUS_TIMEOUT_FULL))) break;
          tc_fence_after();
          const uint32_t sa = smem_u32(smem + stage * stage_bytes);
          const uint64_t da = make_smem_desc_sw128(sa, 16, 1024);
          const uint64_t db = make_smem_desc_sw128(sa + MG_A_BYTES, 16, 1024);
#pragma unroll
          for (int k = 0; k < MG_K / 16; ++k)
            umma_f16_ss(d_tmem, da + (uint64_t)(2 * k), db + (uint64_t)(2 * k), idesc, (kb | k) != 0 ? 1u : 0u);
          umma_commit(&empty_bar[stage]);
          if (++stage == p.stages) {
            stage = 0;
            phase ^= 1;
          }
        }
        if (!ok) break;
        umma_commit(&tmem_full[acc]);
        if (++acc == 2) {
          acc = 0;
          acc_phase ^= 1;
        }
      }
    }
  } else {
    const int quarter = warp & 3;
    int acc = 0;
    uint32_t acc_phase = 0;
    for (int tile = blockIdx.x; tile < num_tiles; tile += gridDim.x) {
      const int ti = tile / num_f, f0 = (tile % num_f) * MG_M;
      const long long row0 = p.tile_row[ti];
      if (!mbar_wait_bounded(&tmem_full[acc], acc_phase, abort_flag, p.status, STATUS_TIMEOUT_TMEM_FULL)) break;
      tc_fence_after();
      const uint32_t taddr = tmem_base + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(acc * p.tile);
      const int f = f0 + quarter * 32 + lane;       // this lane's feature
      const int fp = f & ~1;                        // feature pair it stores: even lanes token c, odd lanes token c + 1
      __nv_bfloat16* dst = p.out + (row0 + (lane & 1)) * p.ldo + fp;
      if (p.act == 2) {
        const int fo = ((f0 + quarter * 32 + lane) >> 2) * 2;  // pair of results that four lanes make; of 4 tokens, this lane stores one
        if ((f0 + quarter * 32) / 2 < p.ldo) {
          __nv_bfloat16* d2 = p.out + (row0 + (lane & 1) + (lane & 2)) * p.ldo + fo;
          for (int c0 = 0; c0 < p.tile; c0 += 16) {
            uint32_t r[16];
            tmem_ld_32x32b_x16(taddr + (uint32_t)c0, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; i += 4) {
              float y[2];  // of tokens i and i + 2, odd lanes i + 1 and i + 3
#pragma unroll
              for (int k = 0; k < 2; ++k) {
                const float a = __uint_as_float(r[i + 2 * k]), b = __uint_as_float(r[i + 2 * k + 1]);
                const float got = __shfl_xor_sync(0xffffffffu, (lane & 1) ? a : b, 1);
                const float gate = (lane & 1) ? got : a, up = (lane & 1) ? b : got;
                y[k] = f < p.n_out ? __fdividef(gate, 1.f + __expf(-gate)) * up : 0.f;
              }
              const float got = __shfl_xor_sync(0xffffffffu, (lane & 2) ? y[0] : y[1], 2);
              const uint32_t w = (lane & 2) ? pack_bf16x2(got, y[1]) : pack_bf16x2(y[0], got);
              if (fo < p.ldo) *reinterpret_cast<uint32_t*>(d2 + (long long)(c0 + i) * p.ldo) = w;
            }
          }
        }
      } else if (f0 + quarter * 32 < p.ldo) {
        for (int c0 = 0; c0 < p.tile; c0 += 16) {
          uint32_t r[16];
          tmem_ld_32x32b_x16(taddr + (uint32_t)c0, r);
          tmem_ld_wait();
          float v[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            float x = f < p.n_out ? __uint_as_float(r[i]) : 0.f;
            if (p.act == 1) {
              x = fmaxf(x, 0.f);
              x *= x;
            }
            v[i] = x;
          }
#pragma unroll
          for (int i = 0; i < 16; i += 2) {
            const float got = __shfl_xor_sync(0xffffffffu, (lane & 1) ? v[i] : v[i + 1], 1);
            const uint32_t w = (lane & 1) ? pack_bf16x2(got, v[i + 1]) : pack_bf16x2(v[i], got);
            if (fp < p.ldo) *reinterpret_cast<uint32_t*>(dst + (long long)(c0 + i) * p.ldo) = w;
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tmem_empty[acc]);
      if (++acc == 2) {
        acc = 0;
        acc_phase ^= 1;
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, tmem_cols);
  }
}

int moe_gemm_tc(const void* in, const void* w, void* out, const int* plan, const int* tile_expert, const int* tile_row, int tile,
                int max_tiles, int n_expert, int n_out, int k, long long ldk, long long ldo, int act, int* status, cudaStream_t s) {
  if (tile < 16 || tile > 256 || (tile & (tile - 1)) || (ldk % 8) || (ldo % 8)) return KVB_ERR_ALIGN;
  if ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15) return KVB_ERR_ALIGN;
  CUtensorMap tmW, tmX;
  const uint64_t dw[2] = {(uint64_t)k, (uint64_t)n_expert * n_out}, dx[2] = {(uint64_t)k, (uint64_t)max_tiles * tile};
  const uint64_t st[1] = {(uint64_t)ldk};
  const uint32_t bw[2] = {MG_K, MG_M}, bx[2] = {MG_K, (uint32_t)tile};
  int rc;
  if ((rc = tmap_bf16(&tmW, w, 2, dw, st, bw))) return rc;
  if ((rc = tmap_bf16(&tmX, in, 2, dx, st, bx))) return rc;
  MgParams p;
  p.out = (__nv_bfloat16*)out; p.plan = plan; p.tile_expert = tile_expert; p.tile_row = tile_row;
  p.tile = tile; p.n_out = n_out; p.k = k; p.act = act; p.ldo = ldo; p.status = status;
  const int stage_bytes = MG_A_BYTES + tile * MG_K * 2;
  p.stages = (MG_SMEM_LIMIT - 2048) / stage_bytes;
  if (p.stages > MG_MAX_STAGES) p.stages = MG_MAX_STAGES;
  const int smem = p.stages * stage_bytes + 1024 + 512;
  static PerDeviceOnce once;
  if (once.first()) cudaFuncSetAttribute(moe_gemm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, MG_SMEM_LIMIT);
  const long long tiles = (long long)max_tiles * ((n_out + MG_M - 1) / MG_M);
  int sms = 0, dev = 0;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  const int ctas = (int)(tiles < sms ? tiles : sms);
  moe_gemm_kernel<<<ctas, MG_THREADS, smem, s>>>(tmW, tmX, p);
  return cudaGetLastError() == cudaSuccess ? KVB_OK : KVB_ERR_LAUNCH;
}

}  // namespace kvb
