// Expert GEMM on the 5th-generation tensor cores: rows sorted by expert (moe_plan), every tile of kTok rows has one expert.
//
//   plain   y[r, f]  = act(x[r, :] . w[e, f, :])                          (down; up of experts without gates: PlainAct)
//   gated   y[r, f]  = act(x[r, :] . w[e, f, :], x[r, :] . w[e, F + f, :])       (gate and up rows of one packed matrix; GateAct)
//
// With many rows the plain form takes two feature tiles per row tile, as the gated form does by nature: a tile of x is loaded
// once for both, which is what keeps the loads from L2 below the tensor cores' pace.
//
// Operands are swapped as in the decode GEMM: the UMMA's 128-row side is a tile of 128 weight rows and the rows of x ride
// the N side, so a tile holds 16 to 128 of them and few tokens per expert waste no tensor work.  One CTA per SM walks the
// (feature tile, row tile) pairs, row tiles fastest: CTAs that run at the same time share an expert's weight tiles in L2.  The TMA
// ring does not drain between tiles, and tensor memory holds two accumulator sets, so the epilogue of a tile overlaps the
// main loop of the next.  The number of row tiles in use and their experts are read on the device (no host round trip, a
// captured graph serves every routing).
//
// Warp roles (192 threads): warp 0 = TMA producer, warp 1 = TMEM owner + UMMA issuer, warps 2..5 = epilogue (TMEM lane =
// feature, column = row of x).  All waits are bounded (ptx.cuh).
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kGFeat = 128, kGK = 64, kGThreads = 192;
enum GroupedMode { kGPlain = 0, kGGated = 1, kGPlainPair = 2 };

template <int kTok, int kMode>
struct GroupedCfg {
  static constexpr int kABytes = kGFeat * kGK * 2;
  static constexpr int kBBytes = kTok * kGK * 2;
  static constexpr int kNumA = kMode == kGPlain ? 1 : 2;
  static constexpr int kTileFeat = kMode == kGPlainPair ? 2 * kGFeat : kGFeat;      // output features per tile
  static constexpr int kStageBytes = kNumA * kABytes + kBBytes;
  static constexpr int kStagesRaw = (200 * 1024) / kStageBytes;
  static constexpr int kStages = kStagesRaw > 10 ? 10 : kStagesRaw;
  static constexpr int kAccCols = kTok * kNumA;
  static constexpr int kTmemCols = 2 * kAccCols <= 32 ? 32 : 2 * kAccCols <= 64 ? 64 : 2 * kAccCols <= 128 ? 128 : 2 * kAccCols <= 256 ? 256 : 512;
  static constexpr int kSmemBytes = kStages * kStageBytes + 1024 + 256;
  static_assert(kTok % 16 == 0 && kTok <= 128 && 2 * kAccCols <= 512, "UMMA N and tensor memory");
};

template <int kTok, int kMode>
__global__ void __launch_bounds__(kGThreads, 1)
grouped_gemm_kernel(const __grid_constant__ CUtensorMap tm_x, const __grid_constant__ CUtensorMap tm_w, bf16* __restrict__ out,
                    int ldo, int n_out, int w_rows, int K, const int* __restrict__ tile_expert, const int* __restrict__ num_tiles,
                    int max_tiles, int act, float limit, unsigned* status) {
  using Cfg = GroupedCfg<kTok, kMode>;
  constexpr bool kTwo = Cfg::kNumA == 2, kGated = kMode == kGGated;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + Cfg::kStages * Cfg::kStageBytes);
  uint64_t* empty_bar = full_bar + Cfg::kStages;
  uint64_t* acc_full = empty_bar + Cfg::kStages;       // [2]
  uint64_t* acc_empty = acc_full + 2;                  // [2], one arrival per epilogue warp
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0 && lane == 0) {
    prefetch_tensormap(&tm_x);
    prefetch_tensormap(&tm_w);
    for (int s = 0; s < Cfg::kStages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(&acc_full[b], 1);
      mbar_init(&acc_empty[b], 4);
    }
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, Cfg::kTmemCols);
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  pdl_wait();

  const int row_tiles = min(num_tiles[0], max_tiles);
  const int feat_tiles = (n_out + Cfg::kTileFeat - 1) / Cfg::kTileFeat;
  const int total = row_tiles * feat_tiles;
  const int num_kb = (K + kGK - 1) / kGK;

  if (warp == 0) {
    if (lane == 0) {
      int s = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
        const int rt = tile % row_tiles, f0 = (tile / row_tiles) * Cfg::kTileFeat;
        const int wrow = max(tile_expert[rt], 0) * w_rows + f0;
        const bool two = kGated || (kTwo && f0 + kGFeat < n_out);          // the last pair of feature tiles may be half a pair
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!mbar_wait_parked(&empty_bar[s], ph ^ 1, status)) { ok = false; break; }
          uint8_t* st = smem + s * Cfg::kStageBytes;
          mbar_expect_tx(&full_bar[s], Cfg::kStageBytes - (kTwo && !two ? Cfg::kABytes : 0));
          tma_load_2d(st, &tm_w, &full_bar[s], kb * kGK, wrow);
          if (two) tma_load_2d(st + Cfg::kABytes, &tm_w, &full_bar[s], kb * kGK, wrow + (kGated ? n_out : kGFeat));
          tma_load_2d(st + Cfg::kNumA * Cfg::kABytes, &tm_x, &full_bar[s], kb * kGK, rt * kTok);
          if (++s == Cfg::kStages) { s = 0; ph ^= 1; }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc(kGFeat, kTok, 1, 1);
      int s = 0, n = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x, ++n) {
        const int b = n & 1;
        if (!mbar_wait_parked(&acc_empty[b], ((n >> 1) & 1) ^ 1, status)) break;
        tcgen05_fence_after();
        const uint32_t acc = tmem_base + b * Cfg::kAccCols;
        const bool two = kGated || (kTwo && (tile / row_tiles) * Cfg::kTileFeat + kGFeat < n_out);
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!mbar_wait_parked(&full_bar[s], ph, status)) { ok = false; break; }
          tcgen05_fence_after();
          const uint32_t a_addr = smem_u32(smem + s * Cfg::kStageBytes);
          const uint32_t b_addr = a_addr + Cfg::kNumA * Cfg::kABytes;
#pragma unroll
          for (int k = 0; k < kGK / 16; ++k) {
            umma_f16(acc, umma_desc_k_sw128(a_addr + k * 32), umma_desc_k_sw128(b_addr + k * 32), idesc, (kb | k) != 0);
            if (two)
              umma_f16(acc + kTok, umma_desc_k_sw128(a_addr + Cfg::kABytes + k * 32), umma_desc_k_sw128(b_addr + k * 32), idesc, (kb | k) != 0);
          }
          umma_commit(&empty_bar[s]);
          if (++s == Cfg::kStages) { s = 0; ph ^= 1; }
        }
        if (!ok) break;
        umma_commit(&acc_full[b]);
      }
    }
  } else {
    const int quad = warp & 3;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    int n = 0;
    for (int tile = blockIdx.x; tile < total; tile += gridDim.x, ++n) {
      const int b = n & 1;
      const int rt = tile % row_tiles, f = (tile / row_tiles) * Cfg::kTileFeat + quad * 32 + lane;
      if (!mbar_wait(&acc_full[b], (n >> 1) & 1, status)) break;
      tcgen05_fence_after();
      const uint32_t acc = tmem_base + lane_addr + b * Cfg::kAccCols;
      bf16* dst = out + static_cast<size_t>(rt) * kTok * ldo + f;
      constexpr int kChunk = kTok < 32 ? 16 : 32;
#pragma unroll 1
      for (int c = 0; c < kTok; c += kChunk) {
        uint32_t g[kChunk], u[kChunk];
        if constexpr (kChunk == 32) {
          tmem_ld_x32(acc + c, g);
          if (kTwo) tmem_ld_x32(acc + kTok + c, u);
        } else {
          tmem_ld_x16(acc + c, g);
          if (kTwo) tmem_ld_x16(acc + kTok + c, u);
        }
        tmem_ld_wait();
        if (c + kChunk >= kTok) {                         // the accumulators are in registers: the set may be filled again
          tcgen05_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&acc_empty[b]);
        }
        if (!kGated && act != kPlainNone) {
#pragma unroll
          for (int j = 0; j < kChunk; ++j) {
            g[j] = __float_as_uint(plain_act<false>(act, __uint_as_float(g[j])));
            if (kTwo) u[j] = __float_as_uint(plain_act<false>(act, __uint_as_float(u[j])));
          }
        }
        if (f < n_out) {
#pragma unroll
          for (int j = 0; j < kChunk; ++j) {
            float v = __uint_as_float(g[j]);
            if (kGated) v = gated_act<false>(act, limit, v, __uint_as_float(u[j]));
            dst[static_cast<size_t>(c + j) * ldo] = __float2bfloat16_rn(v);
          }
        }
        if (kMode == kGPlainPair && f + kGFeat < n_out) {
#pragma unroll
          for (int j = 0; j < kChunk; ++j) dst[static_cast<size_t>(c + j) * ldo + kGFeat] = __float2bfloat16_rn(__uint_as_float(u[j]));
        }
      }
    }
  }

  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_base, Cfg::kTmemCols);
  }
}

extern "C" int forge_make_tmap_2d(CUtensorMap* tm, const void* base, uint64_t rows, uint64_t cols, uint64_t ld,
                                  uint32_t box_rows, int elem_bytes);

template <int kTok, int kMode>
static int launch_grouped(const void* x, const void* w, void* out, int experts, int n_out, int K, const int* tile_expert, const int* num_tiles,
                          int max_tiles, int act, float limit, unsigned* status, cudaStream_t stream) {
  using Cfg = GroupedCfg<kTok, kMode>;
  const int w_rows = kMode == kGGated ? 2 * n_out : n_out;
  CUtensorMap tm_x, tm_w;
  if (forge_make_tmap_2d(&tm_x, x, static_cast<uint64_t>(max_tiles) * kTok, K, K, kTok, 2) != 0) return -2;
  if (forge_make_tmap_2d(&tm_w, w, static_cast<uint64_t>(experts) * w_rows, K, K, kGFeat, 2) != 0) return -2;
  auto kern = grouped_gemm_kernel<kTok, kMode>;
  FORGE_ENSURE_DYN_SMEM(kern, Cfg::kSmemBytes);
  const long long tiles = static_cast<long long>(max_tiles) * ((n_out + Cfg::kTileFeat - 1) / Cfg::kTileFeat);
  const int grid = tiles < device_sm_count() ? static_cast<int>(tiles) : device_sm_count();
  return launch_kernel(kern, dim3(grid), dim3(kGThreads), Cfg::kSmemBytes, stream, 0, tm_x, tm_w, static_cast<bf16*>(out), n_out, n_out,
                       w_rows, K, tile_expert, num_tiles, max_tiles, act, limit, status) == cudaSuccess ? 0 : -5;
}

// x [max_tiles * tile, K] bf16, w [experts, n_out or 2 n_out (gated), K], out [max_tiles * tile, n_out]; K a multiple of 8.
extern "C" int forge_grouped_gemm(const void* x, const void* w, void* out, int experts, int n_out, int K, int gated, int tile, int act,
                                  float limit, const int* tile_expert, const int* num_tiles, int max_tiles, unsigned* status, cudaStream_t stream) {
  if (max_tiles <= 0 || n_out <= 0 || K <= 0) return 0;
  if ((K & 7) || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(w) & 15)) return -1;
  if (static_cast<long long>(experts) * n_out * 2 >= (1ll << 31)) return -1;
#define FORGE_G(TOK, PLAIN)                                                                                                       \
  case TOK:                                                                                                                       \
    return gated ? launch_grouped<TOK, kGGated>(x, w, out, experts, n_out, K, tile_expert, num_tiles, max_tiles, act, limit, status, stream)  \
                 : launch_grouped<TOK, PLAIN>(x, w, out, experts, n_out, K, tile_expert, num_tiles, max_tiles, act, limit, status, stream);
  switch (tile) {
    FORGE_G(16, kGPlain)
    FORGE_G(32, kGPlain)
    FORGE_G(64, kGPlainPair)
    FORGE_G(128, kGPlainPair)
  }
#undef FORGE_G
  return -6;
}

}  // namespace forge
