// Attention of prompts over a sliding window on the 5th-generation tensor cores: variable length, grouped queries, keys and
// values read from the paged cache, key and value heads of different width (multiples of 8 up to 256).
//
//   S = Q K^T   K-major boxes of 64 columns; q rows are zero-padded to whole boxes, TMA fills the missing key columns with zeros
//   O += P V    P = softmax weights in fp32, as bf16 hi + lo halves (two products: 16 mantissa bits) that take the place of S in
//               tensor memory, V as TMA delivers it (rows = keys, MN-major)
//
// CTA = 128 query rows of one (sequence, head), key tiles of 64 from the tile that holds the first row's oldest visible key to
// the tile of the last row's own.  A row may see nothing of its CTA's first tiles: its reference maximum is set by the first
// key it does see, and nothing of O needs scaling then.  Warp roles, double-buffered S, the reference maximum that is only
// raised when it has grown by 2^8, and bounded waits as in prefill_umma.cu.  V is double-buffered where that leaves room for two CTAs per
// SM (whose softmax warps hide each other's latency), else single-buffered, else as shared memory allows.
// Options (chunks, bounded scores, sinks, gated output): attend_options.cuh.  Pooled blocks behind the window (pooled.cuh), gathered by
// pool_blocks, are key tiles ahead of the others.
#include "../include/attend_options.cuh"
#include "../include/launch.cuh"
#include "../include/pooled.cuh"
#include "../include/scalar.cuh"

#include <type_traits>

namespace forge {

constexpr int kXM = 128, kXN = 64, kXThreads = 192;
constexpr int kXQBox = kXM * 128;           // bytes of a 128-row x 64-column box
constexpr int kXKBox = kXN * 128;           // bytes of a 64-row x 64-column box

__device__ __forceinline__ uint64_t windowed_desc_mn(uint32_t smem_addr, uint32_t mn_block_bytes) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>((mn_block_bytes >> 4) & 0x3FFFu) << 16;   // next 64 elements along MN
  d |= static_cast<uint64_t>(1024 >> 4) << 32;                         // next 8 rows along K
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;                                 // SWIZZLE_128B
  return d;
}

// Bounded scores: none; by an odd polynomial, where no score of the tile passes the bound before it is applied (|z| <= 1 in
// cap tanh(z)), which is nearly always; by the exponential.  The exponential and the reciprocal of tanh would take three times the
// special-function slots of the softmax itself.
enum { kCapNone, kCapPoly, kCapExp };

struct CapFactors {
  float z, pre, post, c[7];   // z = raw * z; softcap_log2(raw, pre, post) = z (c0 + c1 z^2 + ...)
};

template <int kCap>
__device__ __forceinline__ float windowed_exponent(float raw, float scale_log2, const CapFactors& f, float m_ref) {
  if constexpr (kCap == kCapPoly) {
    const float z = raw * f.z, t = z * z;
    float y = f.c[6];
#pragma unroll
    for (int i = 5; i >= 0; --i) y = fmaf(y, t, f.c[i]);
    return fmaf(z, y, -m_ref);
  } else if constexpr (kCap == kCapExp) {
    return softcap_log2(raw, f.pre, f.post) - m_ref;
  } else {
    return fmaf(raw, scale_log2, -m_ref);
  }
}

// The scores of a tile are read from tensor memory twice, a few columns at a time: the loops stay short enough for the instruction
// caches (unrolled over 64 columns, half of the issue slots went by waiting for instructions).
constexpr int kXCols = 16;

// Maximum of a row's scores over the keys kbase + i in [lo, limit) (kMasked) or all of the tile; `size`: the largest |score|, masked or not.
template <bool kMasked, bool kSize>
__device__ __forceinline__ float windowed_row_max(uint32_t s_addr, int kbase, int lo, int limit, float& size) {
  float m[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY}, a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 1
  for (int c = 0; c < kXN; c += 32) {
    uint32_t v[32];
    tmem_ld_x32(s_addr + c, v);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      const float x = __uint_as_float(v[i]);
      const int key = kbase + c + i;
      m[i & 3] = fmaxf(m[i & 3], (!kMasked || (key >= lo && key < limit)) ? x : -INFINITY);
      if (kSize) a[i & 3] = fmaxf(a[i & 3], fabsf(x));
    }
  }
  size = fmaxf(fmaxf(a[0], a[1]), fmaxf(a[2], a[3]));
  return fmaxf(fmaxf(m[0], m[1]), fmaxf(m[2], m[3]));
}

// p = 2^(s scale - m_ref) of one row, in place of its scores in tensor memory: the 16 columns of 16 keys take 8 columns of hi halves, then
// 8 of lo halves, each an A operand of 16 entries.  Returns the row sum.
template <bool kMasked, int kCap>
__device__ __forceinline__ float windowed_probs(uint32_t s_addr, int kbase, int lo, int limit, float scale_log2, const CapFactors& cap, float m_ref) {
  float ps[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 1
  for (int c = 0; c < kXN; c += kXCols) {
    uint32_t v[kXCols], w[kXCols];
    tmem_ld_x16(s_addr + c, v);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < kXCols; i += 2) {
      const int key = kbase + c + i;
      float p0 = ex2_approx(windowed_exponent<kCap>(__uint_as_float(v[i]), scale_log2, cap, m_ref));
      float p1 = ex2_approx(windowed_exponent<kCap>(__uint_as_float(v[i + 1]), scale_log2, cap, m_ref));
      if (kMasked) {
        p0 = key >= lo && key < limit ? p0 : 0.f;
        p1 = key + 1 >= lo && key + 1 < limit ? p1 : 0.f;
      }
      ps[(i >> 1) & 3] += p0 + p1;
      const uint32_t h = pack_bf16x2(p0, p1);
      w[i >> 1] = h;
      w[8 + (i >> 1)] = pack_bf16x2(p0 - bf16_lo(h), p1 - bf16_hi(h));
    }
    tmem_st_x16(s_addr + c, w);
  }
  return (ps[0] + ps[1]) + (ps[2] + ps[3]);
}

struct WindowedPrefill {
  int H, G, d, dv, nq, nv, v_bufs;          // nq, nv: boxes of 64 columns of keys and of values
  int window, block_size, table_width, num_blocks;
  long long ldo;
  float scale_log2, out_scale;
  CapFactors cap;
  AttendOptions<bf16> opt;
  const int* pool_rows;                     // [seqs] first gathered entry of a sequence
  int pool;                                 // tokens of a block; 0: no pooled blocks
};

// tm_q: [tokens, H * 64 nq], box 128 x 64; tm_k / tm_v: [blocks * G * block_size, d / dv], tm_pk / tm_pv: [entries, G d / G dv], box 64 x 64.
// kOptions 0: none; 1: chunks, sinks, gates; 2: these and bounded scores.  kPool: pooled blocks behind the window.
template <int kOptions, bool kPool>
__global__ void __launch_bounds__(kXThreads, 2)
windowed_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                        const __grid_constant__ CUtensorMap tm_pk, const __grid_constant__ CUtensorMap tm_pv, const int* __restrict__ cu_q, const int* __restrict__ context_lens, const int* __restrict__ tables,
                        bf16* __restrict__ out, const WindowedPrefill z, unsigned* status) {
  constexpr bool kCap = kOptions == 2;
  extern __shared__ __align__(1024) uint8_t smem[];   // the swizzled boxes start on multiples of 1024 bytes
  const uint32_t k_stage = z.nq * kXKBox, v_stage = z.nv * kXKBox;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + z.nq * kXQBox;                   // [2 stages]
  uint8_t* sV = sK + 2 * k_stage;                     // [v_bufs]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + z.v_bufs * v_stage);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = bars + 3;
  uint64_t* v_full = bars + 5;
  uint64_t* v_empty = bars + 7;
  uint64_t* s_full = bars + 9;
  uint64_t* p_full = bars + 11;                       // one arrival per softmax warp
  uint64_t* pv_done = bars + 13;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);

  pdl_launch_dependents();
  pdl_wait();
  if (smem_u32(smem) & 1023) {
    if (threadIdx.x == 0) set_status(status, kStatusBadShape);
    return;
  }
  const int seq = blockIdx.z, h = blockIdx.y, g = h / (z.H / z.G);
  const int q_begin = cu_q[seq], q_len = cu_q[seq + 1] - q_begin;
  const int k_len = min(context_lens[seq], z.table_width * z.block_size);
  const int m0 = (gridDim.x - 1 - blockIdx.x) * kXM;  // late tiles, which see more keys, first
  if (m0 >= q_len) return;                            // uniform for the CTA, before anything is allocated
  const int past = max(k_len - q_len, 0);
  const int kv_end = min(k_len, past + m0 + kXM);
  const int tile0 = oldest_visible(past + m0, z.window, kOptions && z.opt.chunked) / kXN;
  int n_pool = 0;                                     // tiles of pooled blocks: what the CTA's last row sees
  if (kPool) n_pool = (pool_visible(oldest_visible(min(past + q_len, kv_end) - 1, z.window, 0), z.pool) + kXN - 1) / kXN;
  const int n_tiles = n_pool + (kv_end + kXN - 1) / kXN - tile0;
  if (n_tiles <= n_pool) return;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0 && lane == 0) {
    prefetch_tensormap(&tm_q);
    prefetch_tensormap(&tm_k);
    prefetch_tensormap(&tm_v);
    mbar_init(q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
      mbar_init(&s_full[s], 1);
      mbar_init(&p_full[s], 4);
      mbar_init(&pv_done[s], 1);
    }
    fence_mbar_init();
  }
  const uint32_t tmem_cols = z.nv > 2 ? 512 : 256;    // S0 (P0) | S1 (P1) | O
  if (warp == 1) {
    tmem_alloc(tmem_slot, tmem_cols);
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_o = tmem_base + 2 * kXN;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(q_full, z.nq * kXQBox);
      for (int b = 0; b < z.nq; ++b) tma_load_2d(sQ + b * kXQBox, &tm_q, q_full, (h * z.nq + b) * 64, q_begin + m0);
      for (int j = 0; j < n_tiles; ++j) {
        const bool means = kPool && j < n_pool;
        const int s = j & 1, tok = (tile0 + j - n_pool) * kXN;
        const uint32_t ph = (j >> 1) & 1;
        int row, k_col = 0, v_col = 0;
        if (means) {                                                               // columns past a head's are its neighbour's: q is zero there
          row = z.pool_rows[seq] + j * kXN;
          k_col = g * z.d;
          v_col = g * z.dv;
        } else {
          int blk = tables[static_cast<size_t>(seq) * z.table_width + tok / z.block_size];
          if (blk < 0 || blk >= z.num_blocks) {
            set_status(status, kStatusBadIndex);
            blk = 0;
          }
          row = (blk * z.G + g) * z.block_size + tok % z.block_size;               // a tile never straddles a block
        }
        const CUtensorMap* map_k = means ? &tm_pk : &tm_k;
        const CUtensorMap* map_v = means ? &tm_pv : &tm_v;
        if (!mbar_wait_parked(&k_empty[s], ph ^ 1, status)) break;
        mbar_expect_tx(&k_full[s], k_stage);
        for (int b = 0; b < z.nq; ++b) tma_load_2d(sK + s * k_stage + b * kXKBox, map_k, &k_full[s], k_col + b * 64, row);
        const int vs = j % z.v_bufs;
        if (!mbar_wait_parked(&v_empty[vs], ((j / z.v_bufs) & 1) ^ 1, status)) break;
        mbar_expect_tx(&v_full[vs], v_stage);
        for (int b = 0; b < z.nv; ++b) tma_load_2d(sV + vs * v_stage + b * kXKBox, map_v, &v_full[vs], v_col + b * 64, row);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc(kXM, kXN, 1, 1);
      const uint32_t idesc_o = umma_idesc(kXM, z.nv * 64, 1, 1) | (1u << 16);         // B (= V) MN-major
      const uint32_t q_addr = smem_u32(sQ);
      const int steps = (z.d + 15) >> 4;
      bool ok = mbar_wait(q_full, 0, status);
      auto issue_s = [&](int j) -> bool {
        const int s = j & 1;
        if (!mbar_wait_parked(&k_full[s], (j >> 1) & 1, status)) return false;
        // P V of tile j - 2 has read these columns
        if (j >= 2 && !mbar_wait_parked(&pv_done[s], ((j - 2) >> 1) & 1, status)) return false;
        tcgen05_fence_after();
        const uint32_t k_addr = smem_u32(sK + s * k_stage);
        for (int k = 0; k < steps; ++k)
          umma_f16(tmem_base + s * kXN, umma_desc_k_sw128(q_addr + (k >> 2) * kXQBox + (k & 3) * 32),
                   umma_desc_k_sw128(k_addr + (k >> 2) * kXKBox + (k & 3) * 32), idesc_s, k != 0);
        umma_commit(&s_full[s]);
        umma_commit(&k_empty[s]);
        return true;
      };
      ok = ok && issue_s(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (j + 1 < n_tiles) ok = issue_s(j + 1);
        if (!ok) break;
        const int s = j & 1, vs = j % z.v_bufs;
        const uint32_t ph = (j >> 1) & 1;
        if (!mbar_wait_parked(&v_full[vs], (j / z.v_bufs) & 1, status) || !mbar_wait_parked(&p_full[s], ph, status)) {
          ok = false;
          break;
        }
        tcgen05_fence_after();
        const uint32_t v_addr = smem_u32(sV + vs * v_stage);
        const uint32_t p_addr = tmem_base + s * kXN;
#pragma unroll
        for (int k = 0; k < kXN / 16; ++k) {
          const uint64_t vd = windowed_desc_mn(v_addr + k * 16 * 128, kXKBox);
          umma_f16_ts(tmem_o, p_addr + k * 16, vd, idesc_o, (j | k) != 0);
          umma_f16_ts(tmem_o, p_addr + k * 16 + 8, vd, idesc_o, 1);
        }
        umma_commit(&pv_done[s]);
        umma_commit(&v_empty[vs]);
      }
    }
  } else {
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const int qpos = past + m0 + r;
    const int key_limit = min(qpos + 1, k_len), key_lo = oldest_visible(qpos, z.window, kOptions && z.opt.chunked);  // visible keys
    const int block_limit = kPool ? pool_visible(key_lo, z.pool) : 0;                                              // visible blocks
    const int o_cols = z.nv * 64;
    float m_ref = 0.f, l_run = 0.f;
    bool seen = false, ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      ok = mbar_wait(&s_full[j & 1], (j >> 1) & 1, status);
      if (!ok) break;
      tcgen05_fence_after();
      const uint32_t s_addr = tmem_base + lane_addr + (j & 1) * kXN;
      const bool means = kPool && j < n_pool;
      const int kbase = means ? j * kXN : (tile0 + j - n_pool) * kXN;
      const int lo = means ? 0 : key_lo, limit = means ? block_limit : key_limit;            // visible in this tile: [lo, limit)
      const bool masked = !__all_sync(0xffffffffu, kbase >= lo && kbase + kXN <= limit);
      float size;
      float mt = masked ? windowed_row_max<true, kCap>(s_addr, kbase, lo, limit, size) : windowed_row_max<false, kCap>(s_addr, kbase, lo, limit, size);
      mt = kCap && mt != -INFINITY ? softcap_log2(mt, z.cap.pre, z.cap.post) : mt * z.scale_log2;      // scale > 0: both keep the order
      if (!seen && mt != -INFINITY) {                    // nothing of this row is in O yet, or only zeros
        m_ref = mt;
        seen = true;
      }
      if (j > 0) {
        const bool grow = seen && mt - m_ref > 8.f;
        if (__any_sync(0xffffffffu, grow)) {
          ok = mbar_wait(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1, status);
          if (!ok) break;
          tcgen05_fence_after();
          const float m_new = seen ? fmaxf(m_ref, mt) : m_ref;
          const float alpha = exp2f(m_ref - m_new);
#pragma unroll 1
          for (int c = 0; c < o_cols; c += 32) {
            uint32_t o[32];
            tmem_ld_x32(tmem_o + lane_addr + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st_x32(tmem_o + lane_addr + c, o);
          }
          tmem_st_wait();
          tcgen05_fence_before();
          l_run *= alpha;
          m_ref = m_new;
        }
      }
      auto probs = [&](auto masked_c, auto cap_c) {
        return windowed_probs<decltype(masked_c)::value, decltype(cap_c)::value>(s_addr, kbase, lo, limit, z.scale_log2, z.cap, m_ref);
      };
      auto either = [&](auto cap_c) { return masked ? probs(std::true_type{}, cap_c) : probs(std::false_type{}, cap_c); };
      if constexpr (kCap) {
        const bool small = __all_sync(0xffffffffu, size * z.cap.z <= 1.f);
        l_run += small ? either(std::integral_constant<int, kCapPoly>{}) : either(std::integral_constant<int, kCapExp>{});
      } else {
        l_run += either(std::integral_constant<int, kCapNone>{});
      }
      tmem_st_wait();
      tcgen05_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[j & 1]);
    }
    if (ok) ok = mbar_wait(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1, status);
    if (ok) {
      tcgen05_fence_after();
      float top = m_ref;
      if (kOptions && z.opt.sink != nullptr) {                       // one more score, of the denominator alone
        const float sink = z.opt.sink[h] * 1.4426950408889634f;
        top = fmaxf(m_ref, sink);
        l_run = fmaf(l_run, exp2f(m_ref - top), exp2f(sink - top));
      }
      const bool store = m0 + r < q_len;
      float inv = l_run > 0.f ? z.out_scale * exp2f(m_ref - top) / l_run : 0.f;
      const bf16* gate = !kOptions || z.opt.gate == nullptr || !store ? nullptr : z.opt.gate + static_cast<size_t>(q_begin + m0 + r) * z.opt.ldg + static_cast<size_t>(h) * z.opt.gate_head;
      if (gate != nullptr && z.opt.gate_col == 0) {      // one gate per head
        inv *= sigmoid_t<bf16>(load_f(gate));
        gate = nullptr;
      }
      bf16* dst = out + static_cast<size_t>(q_begin + m0 + r) * z.ldo + static_cast<size_t>(h) * z.dv;
#pragma unroll 1
      for (int c = 0; c < o_cols; c += 32) {
        uint32_t o[32];
        tmem_ld_x32(tmem_o + lane_addr + c, o);
        tmem_ld_wait();
        if (store) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c + i >= z.dv) continue;                 // dv is a multiple of 8
            float f[8];
            if (gate != nullptr) load_n<8>(gate + c + i, f);
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(o[i + e]) * inv * (gate != nullptr ? sigmoid_t<bf16>(f[e]) : 1.f);
            store_n<8>(dst + c + i, f);
          }
        }
      }
    }
  }

  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_base, tmem_cols);
  }
}

static CapFactors cap_factors(float scale, float cap) {
  CapFactors f = {};
  if (cap > 0.f) {
    // tanh(z) / z over z^2 <= 1: weighted least squares, refitted until the largest error of tanh was even (7e-8 in fp32)
    constexpr float c[7] = {0.9999997020f, -0.3333213031f, 0.1331958175f, -0.0532657616f, 0.0199731588f, -0.0059511801f, 0.0009637412f};
    f.z = scale / cap;
    f.post = cap * 1.4426950408889634f;
    f.pre = 2.f * 1.4426950408889634f * f.z;
    for (int i = 0; i < 7; ++i) f.c[i] = f.post * c[i];
  }
  return f;
}

static int windowed_prefill_smem(int nq, int nv, int v_bufs) { return nq * (kXQBox + 2 * kXKBox) + v_bufs * nv * kXKBox + 256; }

// Columns of one head's padded query row, or 0 when the kernel does not take these sizes (else: windowed_attend_any).
extern "C" int forge_windowed_prefill_qcols(int d, int dv, int block_size) {
  if ((d & 7) || (dv & 7) || d < 8 || dv < 8 || d > 256 || dv > 256 || block_size % kXN) return 0;
  return 64 * ((d + 63) / 64);
}

extern "C" int forge_make_tmap_2d(CUtensorMap* tm, const void* base, uint64_t rows, uint64_t cols, uint64_t ld,
                                  uint32_t box_rows, int elem_bytes);

// q [tokens][H][q_pitch], q_pitch = forge_windowed_prefill_qcols; sequence s has the step's tokens cu_q[s] .. cu_q[s + 1] (its last
// ones) and context_lens[s] keys; out rows of ldo elements (a multiple of 8), 16-byte aligned; a gate per element likewise.  pool: tokens of a
// pooled block (0: none), pool_k / pool_v [pool_entries][G][d / dv] the gathered entries, pool_rows [seqs] where a sequence's begin.
extern "C" int forge_windowed_prefill(const void* q, int tokens, const void* k_cache, const void* v_cache, const int* cu_q, const int* context_lens,
                                      const int* tables, int table_width, int num_blocks, int block_size, void* out, long long ldo, int num_seqs,
                                      int max_q, int H, int G, int d, int dv, int window, float scale, float out_scale, int chunked, float softcap,
                                      const float* sink, const void* gate, long long ldg, int gate_head, int gate_col, const void* pool_k,
                                      const void* pool_v, const int* pool_rows, int pool_entries, int pool, unsigned* status, cudaStream_t stream) {
  if (tokens <= 0 || num_seqs <= 0 || max_q <= 0) return 0;
  const int qcols = forge_windowed_prefill_qcols(d, dv, block_size);
  if (qcols == 0 || num_seqs > 65535 || H > 65535 || H % G || window < 1 || !(scale > 0.f) || (ldo & 7) || (reinterpret_cast<uintptr_t>(out) & 15)) return -1;
  if (static_cast<long long>(num_blocks) * G * block_size >= (1ll << 31)) return -1;
  if (pool < 0 || (pool > 0 && (chunked || pool_entries < 1 || pool_rows == nullptr))) return -1;
  if (gate != nullptr && gate_col != 0 && (gate_col != 1 || ((ldg | gate_head) & 7) || (reinterpret_cast<uintptr_t>(gate) & 15))) return -1;
  const int nq = qcols / 64, nv = (dv + 63) / 64;
  constexpr int kHalf = 113 * 1024, kAll = 227 * 1024;        // two CTAs per SM, one
  int v_bufs = 2;
  if (nv <= 2 && windowed_prefill_smem(nq, nv, 2) > kHalf && windowed_prefill_smem(nq, nv, 1) <= kHalf) v_bufs = 1;
  if (windowed_prefill_smem(nq, nv, v_bufs) > kAll) v_bufs = 1;
  const int smem = windowed_prefill_smem(nq, nv, v_bufs);
  if (smem > kAll) return -1;
  const WindowedPrefill z = {H, G, d, dv, nq, nv, v_bufs, window, block_size, table_width, num_blocks, ldo, scale * 1.4426950408889634f, out_scale,
                             cap_factors(scale, softcap),
                             {chunked, softcap, sink, static_cast<const bf16*>(gate), ldg, gate_head, gate_col}, pool_rows, pool};
  CUtensorMap tm_q, tm_k, tm_v, tm_pk, tm_pv;
  const uint64_t qw = static_cast<uint64_t>(H) * qcols, rows = static_cast<uint64_t>(num_blocks) * G * block_size;
  if (forge_make_tmap_2d(&tm_q, q, tokens, qw, qw, kXM, 2) != 0) return -2;
  if (forge_make_tmap_2d(&tm_k, k_cache, rows, d, d, kXN, 2) != 0) return -2;
  if (forge_make_tmap_2d(&tm_v, v_cache, rows, dv, dv, kXN, 2) != 0) return -2;
  tm_pk = tm_k;
  tm_pv = tm_v;
  if (pool > 0) {
    const uint64_t kw = static_cast<uint64_t>(G) * d, vw = static_cast<uint64_t>(G) * dv;
    if (forge_make_tmap_2d(&tm_pk, pool_k, pool_entries, kw, kw, kXN, 2) != 0) return -2;
    if (forge_make_tmap_2d(&tm_pv, pool_v, pool_entries, vw, vw, kXN, 2) != 0) return -2;
  }
  FORGE_ENSURE_DYN_SMEM((windowed_prefill_kernel<0, false>), 227 * 1024);
  FORGE_ENSURE_DYN_SMEM((windowed_prefill_kernel<1, false>), 227 * 1024);
  FORGE_ENSURE_DYN_SMEM((windowed_prefill_kernel<2, false>), 227 * 1024);
  FORGE_ENSURE_DYN_SMEM((windowed_prefill_kernel<0, true>), 227 * 1024);
  FORGE_ENSURE_DYN_SMEM((windowed_prefill_kernel<1, true>), 227 * 1024);
  FORGE_ENSURE_DYN_SMEM((windowed_prefill_kernel<2, true>), 227 * 1024);
  const int options = softcap > 0.f ? 2 : chunked || sink != nullptr || gate != nullptr ? 1 : 0;
  auto k = pool > 0 ? (options == 2 ? windowed_prefill_kernel<2, true> : options == 1 ? windowed_prefill_kernel<1, true> : windowed_prefill_kernel<0, true>)
                    : (options == 2 ? windowed_prefill_kernel<2, false> : options == 1 ? windowed_prefill_kernel<1, false> : windowed_prefill_kernel<0, false>);
  return launch_kernel(k, dim3((max_q + kXM - 1) / kXM, H, num_seqs), dim3(kXThreads), smem, stream, 0, tm_q, tm_k, tm_v, tm_pk, tm_pv,
                       cu_q, context_lens, tables, static_cast<bf16*>(out), z, status) == cudaSuccess ? 0 : -5;
}

}  // namespace forge
