// Latent attention of single query tokens on the 5th-generation tensor cores, straight over the paged latents
// [blocks][block_size][R + rot].
//
// The queries come folded (W_k^T q | rotated part), so all heads of a token share one key row per cached token (its whole
// latent row) and one value row (the first R entries of the SAME row): a tile of 64 keys is read from memory once and serves
// both products for up to 32 heads.  The keys and latents are the UMMA's 128-row side, the heads ride the N side:
//
//   S^T = K Q^T     A = the key tile as TMA delivers it (K-major boxes of 64 columns; rows 64 .. 127 are whatever follows in
//                   shared memory, their scores are not read: the tensor pipe is far from busy), B = the queries
//   O^T += V^T P^T  A = the same boxes read the other way (MN-major: rows = latent columns), B = the softmax weights.  They are
//                   fp32 and enter as bf16 hi and lo halves side by side on N (16 mantissa bits); hi and lo sums meet at the end
//
// All tiles of the step, sequence by sequence and group of heads by group of heads, are dealt out equally to one CTA per SM: a CTA
// walks over pieces (a whole sequence's tiles, or a part of them) without draining its rings in between.  Whole pieces write their
// result, partial ones leave sums that a second kernel merges.  Lengths are read on the device, so a captured graph serves
// any.  A tile is ceil((R + rot) / 128) units of two boxes; a ring of two tiles' units
// or more keeps loads in flight, and a unit is free again as soon as its 128 latent columns have been multiplied.  The products are
// small (N = 16 .. 64), so issuing them is what costs: S has two issuing warps (even and odd units, an accumulator each, added by
// the softmax), O has one, both S and P are double-buffered, and the softmax of a tile overlaps the scores of the next and the
// sums of the one before.  Warp roles (256 threads): warp 0 = TMA producer, warps 1, 2 = issuers of S (1 owns tensor memory),
// warp 3 = issuer of O, warps 4..7 = softmax: scores go through shared memory to
// change from one key per thread to a share of one head's keys per thread.  O is rescaled only when a head's maximum has grown by
// 2^8.  All waits are bounded (ptx.cuh).
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kLdKeys = 64, kLdThreads = 256, kLdBox = kLdKeys * 128, kLdUnit = 2 * kLdBox, kLdMaxD = 576;

struct LatentDecodeArgs {
  const int* block_tables;   // [seqs][table_width]
  const int* lens;           // [seqs] keys visible, the token's own included
  bf16* o;                   // [seqs][heads][R]
  float* part_o;             // [CTAs][2][N][R]: slot 0 = a piece that starts inside a sequence, 1 = one that only ends there
  float* part_ml;            // [CTAs][2][N][2]
  int table_width, num_blocks, block_shift, heads, R, D, seqs, groups, window;
  float scale_log2;
  unsigned* status;
};

constexpr int kLdMaxSeqs = 1024;

// Share of CTA c of G in U tiles: [ld_start(c), ld_start(c + 1)); ld_owner is its inverse.
__device__ __forceinline__ int ld_start(int c, int G, int U) { return static_cast<int>(static_cast<long long>(U) * c / G); }
__device__ __forceinline__ int ld_owner(int u, int G, int U) { return static_cast<int>((static_cast<long long>(u + 1) * G - 1) / U); }
// A sequence's visible keys are [lo, len); its tiles begin with the one that holds key lo.
__device__ __forceinline__ int ld_len(const LatentDecodeArgs& p, int seq) { return max(min(p.lens[seq], p.table_width << p.block_shift), 0); }
__device__ __forceinline__ int ld_lo(const LatentDecodeArgs& p, int len) { return p.window > 0 ? max(len - p.window, 0) : 0; }
__device__ __forceinline__ int ld_tiles(const LatentDecodeArgs& p, int seq) {
  const int len = ld_len(p, seq);
  return (len + kLdKeys - 1) / kLdKeys - ld_lo(p, len) / kLdKeys;
}

// A CTA's walk over its pieces, the same in every warp role.
struct LatentPiece {
  int u, end;                // next tile of the CTA's share, end of the share
  int seq, group;            // of this piece
  int tile, tiles;           // first tile of this piece within the sequence, tiles of the piece
  bool starts, ends;         // the piece holds the sequence's first / last tile
  __device__ bool next(const int* before, int seqs, int groups) {        // before[s]: tiles of the sequences ahead of s, all groups
    if (u >= end) return false;
    int lo = 0, hi = seqs;                                               // before[lo] <= u < before[hi]
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (before[mid] <= u) lo = mid; else hi = mid;
    }
    const int n = (before[lo + 1] - before[lo]) / groups, off = u - before[lo];
    seq = lo;
    group = off / n;
    tile = off % n;
    tiles = min(n - tile, end - u);
    starts = tile == 0;
    ends = tile + tiles == n;
    u += tiles;
    return true;
  }
};

template <int N>
struct LatentDecodeCfg {
  static constexpr int kSlots = N == 16 ? 12 : 10;
  static constexpr int kTPitch = kLdKeys + 4;                        // floats per head of the transposed scores
  static constexpr int kQBytes = (kLdMaxD / 64) * N * 128;
  static constexpr int kTBytes = (N * kTPitch * 4 + 1023) / 1024 * 1024;      // per buffer; also holds the weights: 2N rows x 128 bytes
  static constexpr int kSmem = kSlots * kLdUnit + kQBytes + 2 * kTBytes + 512 + 1024 + 64;
  static_assert(kTBytes >= 2 * N * 128 && kSlots >= 2 * ((kLdMaxD + 127) / 128) && kSmem <= 227 * 1024, "shared memory");
};

// MN-major operand with the 128-byte swizzle: rows of 64 MN elements, 8 K rows 1024 bytes apart, the next 64 MN elements one box on.
__device__ __forceinline__ uint64_t latent_v_desc(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>((kLdBox >> 4) & 0x3FFF) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}

// A bounded wait by a whole warp, and a value that is the same in all its lanes (UMMA operands live in uniform registers).
__device__ __forceinline__ bool warp_wait(uint64_t* bar, uint32_t parity, unsigned* status) {
  return __all_sync(0xffffffffu, mbar_wait_parked(bar, parity, status));
}
__device__ __forceinline__ uint32_t warp_uniform(uint32_t x) { return __shfl_sync(0xffffffffu, x, 0); }

// tm_q: [seqs * heads, D], box N x 64; tm_kv: [blocks * block_size, D], box min(64, block_size) x 64.
template <int N>
__global__ void __launch_bounds__(kLdThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv, const LatentDecodeArgs p) {
  using Cfg = LatentDecodeCfg<N>;
  constexpr int kHeadThreads = 128 / N, kHeadKeys = kLdKeys / kHeadThreads;   // 8 x 8 or 4 x 16
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* ring = smem;
  uint8_t* sQ = ring + Cfg::kSlots * kLdUnit;
  uint8_t* sTP = sQ + Cfg::kQBytes;                     // [2]: scores [N][kTPitch] fp32, then weights
  uint64_t* bars = reinterpret_cast<uint64_t*>(sTP + 2 * Cfg::kTBytes);
  uint64_t* full = bars;                                // [kSlots]
  uint64_t* empty = full + Cfg::kSlots;                 // [kSlots]
  uint64_t* q_full = empty + Cfg::kSlots;
  uint64_t* s_full = q_full + 1;                        // [2]
  uint64_t* s_empty = q_full + 3;                       // [2], one arrival per softmax warp that reads scores (two of them)
  uint64_t* p_full = q_full + 5;                        // [2], one arrival per softmax warp
  uint64_t* pv_done = q_full + 7;                       // [2]: O += of the tile that used this weights' buffer is complete
  uint64_t* o_full = q_full + 9;                        // one phase per piece
  uint64_t* o_empty = q_full + 10;                      // one arrival per softmax warp
  uint64_t* q_empty = q_full + 11;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 12);
  int* s_grow = reinterpret_cast<int*>(tmem_slot + 1);  // [2]: some head's maximum has grown (by tile parity)
  float* s_scale = reinterpret_cast<float*>(s_grow + 3);       // [N]

  pdl_launch_dependents();
  pdl_wait();
  __shared__ int before[kLdMaxSeqs + 1];
  for (int i = threadIdx.x; i < p.seqs; i += kLdThreads) before[i + 1] = ld_tiles(p, i) * p.groups;
  __syncthreads();
  if (threadIdx.x < 32) {                               // running sum, 32 sequences at a time
    int base = 0;
    for (int i0 = 0; i0 < p.seqs; i0 += 32) {
      const int i = i0 + threadIdx.x;
      int v = i < p.seqs ? before[i + 1] : 0;
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const int w = __shfl_up_sync(0xffffffffu, v, off);
        if (threadIdx.x >= off) v += w;
      }
      if (i < p.seqs) before[i + 1] = base + v;
      base += __shfl_sync(0xffffffffu, v, 31);
    }
    if (threadIdx.x == 0) before[0] = 0;
  }
  __syncthreads();
  const int total = before[p.seqs], G = min(static_cast<int>(gridDim.x), total);      // nobody's share is empty
  if (static_cast<int>(blockIdx.x) >= G) return;        // uniform, before anything is allocated
  LatentPiece pc;
  pc.u = ld_start(blockIdx.x, G, total);
  pc.end = ld_start(blockIdx.x + 1, G, total);
  const int boxes = (p.D + 63) >> 6, units = (boxes + 1) >> 1, m_tiles = (p.R + 127) >> 7;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0 && lane == 0) {
    prefetch_tensormap(&tm_q);
    prefetch_tensormap(&tm_kv);
    for (int s = 0; s < Cfg::kSlots; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(q_full, 1);
    mbar_init(q_empty, min(units, 2));
    mbar_init(o_empty, 4);
    for (int b = 0; b < 2; ++b) {
      mbar_init(&s_full[b], min(units, 2));
      mbar_init(&s_empty[b], 2);
      mbar_init(&p_full[b], 4);
      mbar_init(&pv_done[b], 1);
    }
    mbar_init(o_full, 1);
    s_grow[0] = s_grow[1] = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);                         // S: two buffers x two parts of N columns | O: m_tiles x (hi N, lo N) from column 128
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + 128;

  if (warp == 0) {
    if (lane == 0) {
      const int box_rows = min(kLdKeys, 1 << p.block_shift);
      int slot = 0, n_piece = 0;
      uint32_t phase = 1;
      bool ok = true;
      for (; ok && pc.next(before, p.seqs, p.groups); ++n_piece) {
        if (n_piece > 0) ok = mbar_wait_parked(q_empty, (n_piece - 1) & 1, p.status);
        if (!ok) break;
        mbar_expect_tx(q_full, boxes * N * 128);
        for (int b = 0; b < boxes; ++b) tma_load_2d(sQ + b * N * 128, &tm_q, q_full, b * 64, pc.seq * p.heads + pc.group * N);
        const int* table = p.block_tables + static_cast<size_t>(pc.seq) * p.table_width;
        const int len = ld_len(p, pc.seq), tile0 = ld_lo(p, len) / kLdKeys + pc.tile;
        for (int t = 0; t < pc.tiles && ok; ++t) {
          int rows[4];                                  // cache row of every box_rows keys of the tile
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            rows[i] = 0;
            const int key = (tile0 + t) * kLdKeys + i * box_rows;
            if (i * box_rows < kLdKeys && key < len) {  // past the end: any rows will do, their weights are zero
              int blk = table[key >> p.block_shift];
              if (blk < 0 || blk >= p.num_blocks) {
                set_status(p.status, kStatusBadIndex);
                blk = 0;
              }
              rows[i] = (blk << p.block_shift) + (key & ((1 << p.block_shift) - 1));
            }
          }
          for (int u = 0; u < units; ++u) {
            if (!mbar_wait_parked(&empty[slot], phase, p.status)) { ok = false; break; }
            const int nb = min(2, boxes - 2 * u);
            mbar_expect_tx(&full[slot], nb * kLdBox);
            for (int b = 0; b < nb; ++b)
#pragma unroll
              for (int i = 0; i < 4; ++i)
                if (i * box_rows < kLdKeys)
                  tma_load_2d(ring + slot * kLdUnit + b * kLdBox + i * box_rows * 128, &tm_kv, &full[slot], (2 * u + b) * 64, rows[i]);
            if (++slot == Cfg::kSlots) { slot = 0; phase ^= 1; }
          }
        }
      }
    }
  } else if (warp <= 2) {
    const int part = warp - 1;                          // units part, part + 2, ...
    constexpr uint32_t idesc_s = umma_idesc(128, N, 1, 1);
    const uint64_t k_desc = umma_desc_k_sw128(smem_u32(ring)), q_desc = umma_desc_k_sw128(smem_u32(sQ));
    const int steps = (p.D + 15) >> 4;
    int slot0 = 0, t = 0, n_piece = 0;                  // first unit of the tile; tiles and pieces of this CTA so far
    uint32_t phase0 = 0;
    bool ok = part < units;
    for (; ok && pc.next(before, p.seqs, p.groups); ++n_piece) {
      ok = warp_wait(q_full, n_piece & 1, p.status);
      for (int left = pc.tiles; left > 0 && ok; --left, ++t) {
        if (t >= 2) ok = warp_wait(&s_empty[t & 1], ((t >> 1) - 1) & 1, p.status);       // softmax has read S of tile t - 2
        const uint32_t d = warp_uniform(tmem_s + ((t & 1) * 2 + part) * N);
        for (int u = part; u < units && ok; u += 2) {
          int slot = slot0 + u;
          uint32_t phase = phase0;
          if (slot >= Cfg::kSlots) { slot -= Cfg::kSlots; phase ^= 1; }
          ok = warp_wait(&full[slot], phase, p.status);
          if (!ok) break;
          tcgen05_fence_after();
          const uint64_t ad = k_desc + warp_uniform(slot * (kLdUnit >> 4)), bd = q_desc + warp_uniform(u * (2 * N * 128 >> 4));
          const uint32_t more = warp_uniform(u != part);
          const int n = steps - u * 8;
          auto product = [&](int k) {
            umma_f16_warp(d, ad + (((k >> 2) * kLdBox + (k & 3) * 32) >> 4), bd + (((k >> 2) * N * 128 + (k & 3) * 32) >> 4), idesc_s, k != 0 ? 1 : more);
          };
          if (n >= 8) {
#pragma unroll
            for (int k = 0; k < 8; ++k) product(k);
          } else {
#pragma unroll
            for (int k = 0; k < 7; ++k)
              if (k < n) product(k);
          }
          if (u >= m_tiles) umma_commit_warp(&empty[slot]);      // no value columns in this unit
        }
        if (ok) umma_commit_warp(&s_full[t & 1]);
        slot0 += units;
        if (slot0 >= Cfg::kSlots) { slot0 -= Cfg::kSlots; phase0 ^= 1; }
      }
      if (ok) umma_commit_warp(q_empty);
    }
  } else if (warp == 3) {
    constexpr uint32_t idesc_o = umma_idesc(128, 2 * N, 1, 1) | (1u << 15);           // A (= V^T) MN-major
    const uint64_t v_desc = latent_v_desc(smem_u32(ring)), p_desc = umma_desc_k_sw128(smem_u32(sTP));
    int slot0 = 0, t = 0, n_piece = 0;                  // first unit of the tile; tiles and pieces so far
    bool ok = true;
    for (; ok && pc.next(before, p.seqs, p.groups); ++n_piece) {
      if (n_piece > 0) ok = warp_wait(o_empty, (n_piece - 1) & 1, p.status);            // the piece before has been read
      for (int i = 0; i < pc.tiles && ok; ++i, ++t) {
        ok = warp_wait(&p_full[t & 1], (t >> 1) & 1, p.status);    // and with it: the tile's units are in place
        if (!ok) break;
        tcgen05_fence_after();
        const uint64_t bd = p_desc + warp_uniform((t & 1) * (Cfg::kTBytes >> 4));
        int slot = slot0;
        for (int m = 0; m < m_tiles; ++m) {
          const uint32_t d = warp_uniform(tmem_o + m * 2 * N);
          const uint64_t ad = v_desc + warp_uniform(slot * (kLdUnit >> 4));
#pragma unroll
          for (int k = 0; k < kLdKeys / 16; ++k) umma_f16_warp(d, ad + (k * 16 * 128 >> 4), bd + (k * 32 >> 4), idesc_o, k != 0 || i != 0);
          umma_commit_warp(&empty[slot]);
          if (++slot == Cfg::kSlots) slot = 0;
        }
        umma_commit_warp(&pv_done[t & 1]);
        slot0 += units;
        if (slot0 >= Cfg::kSlots) slot0 -= Cfg::kSlots;
      }
      if (ok) umma_commit_warp(o_full);
    }
  } else {
    const int quad = warp & 3, key = quad * 32 + lane;   // TMEM lane = key of the tile
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const int tid = key, head = tid / kHeadThreads, sub = tid % kHeadThreads;
    int t = 0, n_piece = 0;                              // tiles and pieces of this CTA so far
    for (; pc.next(before, p.seqs, p.groups); ++n_piece) {
      const int len = ld_len(p, pc.seq), lo = ld_lo(p, len), tile0 = lo / kLdKeys + pc.tile, h0 = pc.group * N;
      float m_ref = 0.f, l_run = 0.f;
      // a wait that runs out is in the status word; the loop goes on, so that all four warps meet at the barriers
      for (int i_tile = 0; i_tile < pc.tiles; ++i_tile, ++t) {
        mbar_wait_parked(&s_full[t & 1], (t >> 1) & 1, p.status);
        if (t >= 2) mbar_wait_parked(&pv_done[t & 1], ((t >> 1) - 1) & 1, p.status);     // the buffer's weights (tile t - 2) have been used
        tcgen05_fence_after();
        uint8_t* tp = sTP + (t & 1) * Cfg::kTBytes;
        float* sT = reinterpret_cast<float*>(tp);
        if (quad < 2) {
          uint32_t v[N], w[N];
          const uint32_t at = tmem_s + (t & 1) * 2 * N + lane_addr;
          if constexpr (N == 16) {
            tmem_ld_x16(at, v);
            tmem_ld_x16(at + N, w);
          } else {
            tmem_ld_x32(at, v);
            tmem_ld_x32(at + N, w);
          }
          tmem_ld_wait();
          if (units > 1) {
#pragma unroll
            for (int h = 0; h < N; ++h) v[h] = __float_as_uint(__uint_as_float(v[h]) + __uint_as_float(w[h]));
          }
          tcgen05_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&s_empty[t & 1]);
          const int at_key = (tile0 + i_tile) * kLdKeys + key;
          const bool in = at_key >= lo && at_key < len;
#pragma unroll
          for (int h = 0; h < N; ++h) sT[h * Cfg::kTPitch + key] = in ? __uint_as_float(v[h]) * p.scale_log2 : -INFINITY;
        }
        named_barrier_sync(1, 128);
        if (tid == 0) s_grow[(t + 1) & 1] = 0;             // last read in tile t - 1, which everyone has left
        float x[kHeadKeys], mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < kHeadKeys; i += 4) {           // keys 8 (sub + kHeadThreads j) .. + 7: whole 16-byte chunks of the weight rows
          const int at = ((i >> 3) * kHeadThreads + sub) * 8 + (i & 7);
          const float4 f = *reinterpret_cast<const float4*>(sT + head * Cfg::kTPitch + at);
          x[i] = f.x;
          x[i + 1] = f.y;
          x[i + 2] = f.z;
          x[i + 3] = f.w;
          mx = fmaxf(mx, fmaxf(fmaxf(f.x, f.y), fmaxf(f.z, f.w)));
        }
#pragma unroll
        for (int off = kHeadThreads / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        float alpha = 1.f;                                 // mx is finite: a tile holds at least one visible key
        if (i_tile == 0) {
          m_ref = mx;
        } else if (mx - m_ref > 8.f) {
          alpha = exp2f(m_ref - mx);
          m_ref = mx;
          s_grow[t & 1] = 1;
        }
        if (sub == 0) s_scale[head] = alpha;
        l_run *= alpha;
        named_barrier_sync(1, 128);                        // scores are in registers, scales and the flag are set
        if (i_tile > 0 && s_grow[t & 1]) {
          mbar_wait_parked(&pv_done[(t - 1) & 1], ((t - 1) >> 1) & 1, p.status);         // every earlier product has landed in O
          tcgen05_fence_after();
#pragma unroll 1
          for (int c = 0; c < m_tiles * 2 * N; c += 32) {
            uint32_t o[32];
            tmem_ld_x32(tmem_o + lane_addr + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * s_scale[i % N]);
            tmem_st_x32(tmem_o + lane_addr + c, o);
          }
          tmem_st_wait();
        }
#pragma unroll
        for (int i = 0; i < kHeadKeys; i += 8) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float p0 = ex2_approx(x[i + 2 * e] - m_ref), p1 = ex2_approx(x[i + 2 * e + 1] - m_ref);
            l_run += p0 + p1;
            hi[e] = pack_bf16x2(p0, p1);
            lo[e] = pack_bf16x2(p0 - bf16_lo(hi[e]), p1 - bf16_hi(hi[e]));
          }
          const int c = (i >> 3) * kHeadThreads + sub;     // 16-byte chunk of the 64 keys
          uint8_t* row = tp + head * 128 + ((c ^ (head & 7)) << 4);
          *reinterpret_cast<uint4*>(row) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(row + N * 128) = make_uint4(lo[0], lo[1], lo[2], lo[3]);    // N is a multiple of 8: same swizzle phase
        }
        fence_proxy_async_smem();
        tcgen05_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_full[t & 1]);
      }
#pragma unroll
      for (int off = kHeadThreads / 2; off > 0; off >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, off);
      const bool whole = pc.starts && pc.ends;
      const size_t part = static_cast<size_t>(blockIdx.x) * 2 + (pc.starts ? 1 : 0);
      mbar_wait_parked(o_full, n_piece & 1, p.status);     // and with it: every warp is past its last use of s_scale
      if (sub == 0) {
        s_scale[head] = whole ? 1.f / l_run : 1.f;
        if (!whole) {
          p.part_ml[(part * N + head) * 2] = m_ref;
          p.part_ml[(part * N + head) * 2 + 1] = l_run;
        }
      }
      named_barrier_sync(1, 128);
      tcgen05_fence_after();
      for (int m = 0; m < m_tiles; ++m) {
        __syncwarp();
        uint32_t hi[N], lo[N];
        if constexpr (N == 16) {
          tmem_ld_x16(tmem_o + lane_addr + m * 2 * N, hi);
          tmem_ld_x16(tmem_o + lane_addr + m * 2 * N + N, lo);
        } else {
          tmem_ld_x32(tmem_o + lane_addr + m * 2 * N, hi);
          tmem_ld_x32(tmem_o + lane_addr + m * 2 * N + N, lo);
        }
        tmem_ld_wait();
        if (m + 1 == m_tiles) {                            // O is in registers: the next piece may begin
          tcgen05_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(o_empty);
        }
        const int d = m * 128 + key;
        if (d >= p.R) continue;
#pragma unroll
        for (int h = 0; h < N; ++h) {
          const float v = __uint_as_float(hi[h]) + __uint_as_float(lo[h]);
          if (!whole) p.part_o[(part * N + h) * p.R + d] = v;
          else if (h0 + h < p.heads) p.o[(static_cast<size_t>(pc.seq) * p.heads + h0 + h) * p.R + d] = __float2bfloat16_rn(v * s_scale[h]);
        }
      }
      named_barrier_sync(1, 128);                          // s_scale has been read
    }
  }

  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_s, 512);
  }
}

// One CTA per (head, sequence): the partial sums of a sequence whose tiles went to several CTAs, weighted by their maxima.
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentDecodeArgs p, int N, int ctas) {
  __shared__ int red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, seq = blockIdx.y, group = h / N, hg = h % N;
  int mine = 0, all = 0;                               // tiles ahead of this sequence, tiles of the step
  for (int s = threadIdx.x; s < p.seqs; s += 128) {
    const int n = ld_tiles(p, s) * p.groups;
    all += n;
    if (s < seq) mine += n;
  }
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) {
    mine += __shfl_xor_sync(0xffffffffu, mine, off);
    all += __shfl_xor_sync(0xffffffffu, all, off);
  }
  if ((threadIdx.x & 31) == 0) {
    red[threadIdx.x >> 5] = mine;
    red[4 + (threadIdx.x >> 5)] = all;
  }
  __syncthreads();
  const int n = ld_tiles(p, seq), U = red[4] + red[5] + red[6] + red[7], G = min(ctas, U);
  bf16* o = p.o + (static_cast<size_t>(seq) * p.heads + h) * p.R;
  if (n == 0) {                                        // padding of a graph bucket: defined values
    for (int i = threadIdx.x; i < p.R; i += 128) o[i] = __float2bfloat16_rn(0.f);
    return;
  }
  const int first = red[0] + red[1] + red[2] + red[3] + group * n;
  const int c0 = ld_owner(first, G, U), c1 = ld_owner(first + n - 1, G, U);
  if (c0 == c1) return;                                // one piece: already written
  auto part = [&](int c) { return (static_cast<size_t>(c) * 2 + (c == c0 ? 1 : 0)) * N + hg; };
  float m = -INFINITY;
  for (int c = c0; c <= c1; ++c) m = fmaxf(m, p.part_ml[part(c) * 2]);
  float l = 0.f;
  for (int c = c0; c <= c1; ++c) l += p.part_ml[part(c) * 2 + 1] * exp2f(p.part_ml[part(c) * 2] - m);
  const float inv = 1.f / l;
  for (int i = threadIdx.x * 4; i < p.R; i += 128 * 4) {
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c = c0; c <= c1; ++c) {
      const float w = exp2f(p.part_ml[part(c) * 2] - m) * inv;
      const float4 v = *reinterpret_cast<const float4*>(p.part_o + part(c) * p.R + i);
      s.x = fmaf(w, v.x, s.x);
      s.y = fmaf(w, v.y, s.y);
      s.z = fmaf(w, v.z, s.z);
      s.w = fmaf(w, v.w, s.w);
    }
    *reinterpret_cast<uint2*>(o + i) = make_uint2(pack_bf16x2(s.x, s.y), pack_bf16x2(s.z, s.w));
  }
}

extern "C" int forge_make_tmap_2d(CUtensorMap* tm, const void* base, uint64_t rows, uint64_t cols, uint64_t ld,
                                  uint32_t box_rows, int elem_bytes);

// 1 if the kernel takes these sizes (else: latent_attend_any).
extern "C" int forge_latent_decode_ok(int R, int rot, int block_size) {
  return R >= 8 && R <= 512 && R % 8 == 0 && rot % 8 == 0 && R + rot <= kLdMaxD && block_size >= 16 && (block_size & (block_size - 1)) == 0;
}

// Heads a CTA takes, and fp32 elements of scratch for `ctas` CTAs.
static int latent_decode_group(int heads) { return heads > 16 ? 32 : 16; }
extern "C" long long forge_latent_decode_scratch(int heads, int R, int ctas) { return 2ll * ctas * latent_decode_group(heads) * (R + 2); }

template <int N>
static int launch_latent_decode(const CUtensorMap& tm_q, const CUtensorMap& tm_kv, const LatentDecodeArgs& p, int ctas, cudaStream_t stream) {
  auto kern = latent_decode_kernel<N>;
  FORGE_ENSURE_DYN_SMEM(kern, LatentDecodeCfg<N>::kSmem);
  return launch_kernel(kern, dim3(ctas), dim3(kLdThreads), LatentDecodeCfg<N>::kSmem, stream, 0, tm_q, tm_kv, p) == cudaSuccess ? 0 : -2;
}

// qa [seqs][heads][R + rot] bf16; lens = keys per sequence, of which the last `window` are visible (0: all); scratch: forge_latent_decode_scratch floats, 16-byte aligned.
extern "C" int forge_latent_decode(const void* qa, const void* cache, const int* block_tables, const int* lens, void* o, float* scratch,
                                   int ctas, int seqs, int heads, int R, int rot, int table_width, int num_blocks, int block_size,
                                   int window, float scale, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  const int D = R + rot, n = latent_decode_group(heads), groups = (heads + n - 1) / n;
  if (!forge_latent_decode_ok(R, rot, block_size) || seqs > kLdMaxSeqs || ctas < 1 || (reinterpret_cast<uintptr_t>(qa) & 15) ||
      (reinterpret_cast<uintptr_t>(cache) & 15) || (reinterpret_cast<uintptr_t>(scratch) & 15) ||
      static_cast<long long>(num_blocks) * block_size >= (1ll << 31) ||
      static_cast<long long>(seqs) * groups * (static_cast<long long>(table_width) * block_size / kLdKeys + 1) >= (1ll << 31))
    return -1;
  int shift = 0;
  while ((1 << shift) < block_size) ++shift;
  const LatentDecodeArgs p = {block_tables, lens, static_cast<bf16*>(o), scratch, scratch + 2ll * ctas * n * R, table_width, num_blocks, shift,
                              heads, R, D, seqs, groups, window, scale * 1.4426950408889634f, status};
  CUtensorMap tm_q, tm_kv;
  if (forge_make_tmap_2d(&tm_q, qa, static_cast<uint64_t>(seqs) * heads, D, D, n, 2) != 0) return -2;
  if (forge_make_tmap_2d(&tm_kv, cache, static_cast<uint64_t>(num_blocks) * block_size, D, D, block_size < kLdKeys ? block_size : kLdKeys, 2) != 0) return -2;
  const int rc = n == 32 ? launch_latent_decode<32>(tm_q, tm_kv, p, ctas, stream) : launch_latent_decode<16>(tm_q, tm_kv, p, ctas, stream);
  if (rc != 0) return rc;
  return launch_kernel(latent_merge_kernel, dim3(heads, seqs), dim3(128), 0, stream, 0, p, n, ctas) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
