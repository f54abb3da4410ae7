// Latent attention of prompts on the 5th-generation tensor cores.  A prompt's queries see keys and values rebuilt per head:
// the cached latents of the step's sequences are gathered into one contiguous buffer (latent_gather), one GEMM with the packed
// key / value matrices expands them, and the kernel below attends.  Two little kernels put the operands in shape:
//
//   latent_gather     paged rows [c | rotated key part] -> c [keys][R] and k_rot [keys][rot], sequences one after another, of each the
//                     last keys (all that its queries see)
//   latent_pack_q     q [tokens][heads][dim + rot] -> [tokens][heads][Dq]: the rotated part rotated, both parts zero-padded to
//                     multiples of 64 columns, so that a 64-column box of keys may run into its neighbour's columns
//
//   S = Qn Kn^T + Qr Kr^T   K-major boxes of 64 columns; the rotated key part is one box shared by all heads
//   O += P V                P = softmax weights in fp32, as bf16 hi + lo halves (two products: 16 mantissa bits), V as TMA
//                           delivers it (rows = keys, MN-major)
//
// CTA = 128 query rows of one (sequence, head), key tiles of 64.  Warp roles, double-buffered S and P, the reference maximum
// that is only raised when it has grown by 2^8, and bounded waits as in prefill_umma.cu.  With a window the key tiles begin with the one
// that holds the first row's oldest visible key; a row may see nothing of them, as in windowed_prefill.cu.
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kVM = 128, kVN = 64, kVThreads = 192;
constexpr int kVQBox = kVM * 128;           // bytes of a 128-row x 64-column box
constexpr int kVKBox = kVN * 128;           // bytes of a 64-row x 64-column box
constexpr int kVStages = 2;

__device__ __forceinline__ uint64_t latent_desc_mn(uint32_t smem_addr, uint32_t mn_block_bytes) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>((mn_block_bytes >> 4) & 0x3FFFu) << 16;   // next 64 elements along MN
  d |= static_cast<uint64_t>(1024 >> 4) << 32;                         // next 8 rows along K
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;                                 // SWIZZLE_128B
  return d;
}

template <bool kMasked>
__device__ __forceinline__ float latent_row_max(const uint32_t (&v)[kVN], int kbase, int lo, int limit) {
  float m[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
  for (int i = 0; i < kVN; i += 4)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float x = __uint_as_float(v[i + e]);
      m[e] = fmaxf(m[e], (!kMasked || (kbase + i + e >= lo && kbase + i + e < limit)) ? x : -INFINITY);
    }
  return fmaxf(fmaxf(m[0], m[1]), fmaxf(m[2], m[3]));
}

// p = 2^(s scale - m_ref) of one row -> hi and lo bf16 halves in shared memory (K-major, 128-byte swizzle); returns the row sum.
template <bool kMasked>
__device__ __forceinline__ float latent_probs(const uint32_t (&v)[kVN], int kbase, int first, int limit, float scale_log2, float m_ref, uint8_t* p_row,
                                              int r) {
  float ps[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int c = 0; c < kVN; c += 8) {
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int i = 0; i < 8; i += 2) {
      float p0 = ex2_approx(fmaf(__uint_as_float(v[c + i]), scale_log2, -m_ref));
      float p1 = ex2_approx(fmaf(__uint_as_float(v[c + i + 1]), scale_log2, -m_ref));
      if (kMasked) {
        p0 = kbase + c + i >= first && kbase + c + i < limit ? p0 : 0.f;
        p1 = kbase + c + i + 1 >= first && kbase + c + i + 1 < limit ? p1 : 0.f;
      }
      ps[i >> 1] += p0 + p1;
      const uint32_t h = pack_bf16x2(p0, p1);
      hi[i >> 1] = h;
      lo[i >> 1] = pack_bf16x2(p0 - bf16_lo(h), p1 - bf16_hi(h));
    }
    const int at = ((c >> 3) ^ (r & 7)) << 4;
    *reinterpret_cast<uint4*>(p_row + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(p_row + kVQBox + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  return (ps[0] + ps[1]) + (ps[2] + ps[3]);
}

// Boxes of 64 columns: nb1 of the unrotated part, nb2 of the rotated part, nv of the values.
struct LatentPrefillSizes {
  int heads, dim, rot, vdim, nb1, nb2, nv, tok0, window;
};

// tm_q: [tokens, heads * 64 (nb1 + nb2)], box 128 x 64; tm_kv: [keys, heads * (dim + vdim)], tm_r: [keys, rot], box 64 x 64.
__global__ void __launch_bounds__(kVThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv,
                      const __grid_constant__ CUtensorMap tm_r, const int* __restrict__ cu_q, const int* __restrict__ cu_k,
                      bf16* __restrict__ out, const LatentPrefillSizes z, float scale_log2, unsigned* status) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nq = z.nb1 + z.nb2;
  const uint32_t k_stage = nq * kVKBox, v_stage = z.nv * kVKBox;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + nq * kVQBox;                     // [2 stages]
  uint8_t* sV = sK + kVStages * k_stage;              // [2 stages]
  uint8_t* sP = sV + kVStages * v_stage;              // [2][hi, lo]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + 4 * kVQBox);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = bars + 3;
  uint64_t* v_full = bars + 5;
  uint64_t* v_empty = bars + 7;
  uint64_t* s_full = bars + 9;
  uint64_t* s_empty = bars + 11;                      // one arrival per softmax warp
  uint64_t* p_full = bars + 13;                       // one arrival per softmax warp
  uint64_t* pv_done = bars + 15;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 17);

  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, h = blockIdx.y;
  const int q_begin = cu_q[seq], q_len = cu_q[seq + 1] - q_begin;
  const int k_row0 = cu_k[seq], k_len = cu_k[seq + 1] - k_row0;
  const int m_tile = gridDim.x - 1 - blockIdx.x;      // heavy (late) tiles first
  const int m0 = m_tile * kVM;
  if (m0 >= q_len) return;                            // uniform for the CTA, before anything is allocated
  const int past = k_len - q_len;
  const int kv_end = min(k_len, past + m0 + kVM);
  const int tile0 = z.window > 0 ? max(past + m0 - z.window + 1, 0) / kVN : 0;
  const int n_tiles = (kv_end + kVN - 1) / kVN - tile0;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0 && lane == 0) {
    prefetch_tensormap(&tm_q);
    prefetch_tensormap(&tm_kv);
    prefetch_tensormap(&tm_r);
    mbar_init(q_full, 1);
    for (int s = 0; s < kVStages; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
      mbar_init(&s_full[s], 1);
      mbar_init(&s_empty[s], 4);
      mbar_init(&p_full[s], 4);
      mbar_init(&pv_done[s], 1);
    }
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 256);                       // S0 | S1 | O (up to 128 columns)
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_o = tmem_base + 2 * kVN;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(q_full, nq * kVQBox);
      for (int b = 0; b < nq; ++b) tma_load_2d(sQ + b * kVQBox, &tm_q, q_full, (h * nq + b) * 64, q_begin - z.tok0 + m0);
      for (int j = 0; j < n_tiles; ++j) {
        const int s = j & 1, row = k_row0 + (tile0 + j) * kVN;
        const uint32_t ph = (j >> 1) & 1;
        if (!mbar_wait_parked(&k_empty[s], ph ^ 1, status)) break;
        mbar_expect_tx(&k_full[s], k_stage);
        uint8_t* st = sK + s * k_stage;
        for (int b = 0; b < z.nb1; ++b) tma_load_2d(st + b * kVKBox, &tm_kv, &k_full[s], h * z.dim + b * 64, row);
        for (int b = 0; b < z.nb2; ++b) tma_load_2d(st + (z.nb1 + b) * kVKBox, &tm_r, &k_full[s], b * 64, row);
        if (!mbar_wait_parked(&v_empty[s], ph ^ 1, status)) break;
        mbar_expect_tx(&v_full[s], v_stage);
        for (int b = 0; b < z.nv; ++b)
          tma_load_2d(sV + s * v_stage + b * kVKBox, &tm_kv, &v_full[s], z.heads * z.dim + h * z.vdim + b * 64, row);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc(kVM, kVN, 1, 1);
      const uint32_t idesc_o = umma_idesc(kVM, z.nv * 64, 1, 1) | (1u << 16);         // B (= V) MN-major
      const uint32_t q_addr = smem_u32(sQ), p_addr = smem_u32(sP);
      const int steps1 = (z.dim + 15) >> 4, steps2 = (z.rot + 15) >> 4;
      bool ok = mbar_wait(q_full, 0, status);
      auto issue_s = [&](int j) -> bool {
        const int s = j & 1;
        if (!mbar_wait_parked(&k_full[s], (j >> 1) & 1, status)) return false;
        if (!mbar_wait_parked(&s_empty[s], ((j >> 1) & 1) ^ 1, status)) return false; // softmax has read S of tile j - 2
        tcgen05_fence_after();
        const uint32_t k_addr = smem_u32(sK + s * k_stage);
        for (int k = 0; k < steps1 + steps2; ++k) {
          const int box = k < steps1 ? k >> 2 : z.nb1 + ((k - steps1) >> 2), sub = (k < steps1 ? k : k - steps1) & 3;
          umma_f16(tmem_base + s * kVN, umma_desc_k_sw128(q_addr + box * kVQBox + sub * 32),
                   umma_desc_k_sw128(k_addr + box * kVKBox + sub * 32), idesc_s, k != 0);
        }
        umma_commit(&s_full[s]);
        umma_commit(&k_empty[s]);
        return true;
      };
      ok = ok && issue_s(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (j + 1 < n_tiles) ok = issue_s(j + 1);
        if (!ok) break;
        const int s = j & 1;
        const uint32_t ph = (j >> 1) & 1;
        if (!mbar_wait_parked(&v_full[s], ph, status) || !mbar_wait_parked(&p_full[s], ph, status)) {
          ok = false;
          break;
        }
        tcgen05_fence_after();
        const uint32_t v_addr = smem_u32(sV + s * v_stage);
        const uint32_t pj_addr = p_addr + s * 2 * kVQBox;
#pragma unroll
        for (int k = 0; k < kVN / 16; ++k) {
          const uint64_t vd = latent_desc_mn(v_addr + k * 16 * 128, kVKBox);
          umma_f16(tmem_o, umma_desc_k_sw128(pj_addr + k * 32), vd, idesc_o, (j | k) != 0);
          umma_f16(tmem_o, umma_desc_k_sw128(pj_addr + kVQBox + k * 32), vd, idesc_o, 1);
        }
        umma_commit(&pv_done[s]);
        umma_commit(&v_empty[s]);
      }
    }
  } else {
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const int limit = min(past + m0 + r + 1, k_len), lo = z.window > 0 ? past + m0 + r + 1 - z.window : 0;   // visible keys: [lo, limit)
    const int o_cols = z.nv * 64;
    float m_ref = 0.f, l_run = 0.f;
    bool seen = false, ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      ok = mbar_wait(&s_full[j & 1], (j >> 1) & 1, status);
      if (!ok) break;
      tcgen05_fence_after();
      const uint32_t s_addr = tmem_base + lane_addr + (j & 1) * kVN;
      const int kbase = (tile0 + j) * kVN;
      uint32_t v[kVN];
#pragma unroll
      for (int c = 0; c < kVN; c += 32) tmem_ld_x32(s_addr + c, v + c);
      tmem_ld_wait();
      tcgen05_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_empty[j & 1]);
      const bool masked = !__all_sync(0xffffffffu, kbase >= lo && kbase + kVN <= limit);
      float mt = masked ? latent_row_max<true>(v, kbase, lo, limit) : latent_row_max<false>(v, kbase, lo, limit);
      mt *= scale_log2;
      if (!seen && mt != -INFINITY) {                   // nothing of this row is in O yet, or only zeros
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
      if (j >= 2) {                                     // P buffer j & 1 was last read by P V of tile j - 2
        ok = mbar_wait(&pv_done[j & 1], ((j >> 1) - 1) & 1, status);
        if (!ok) break;
      }
      uint8_t* p_row = sP + (j & 1) * 2 * kVQBox + r * 128;
      l_run += masked ? latent_probs<true>(v, kbase, lo, limit, scale_log2, m_ref, p_row, r)
                      : latent_probs<false>(v, kbase, lo, limit, scale_log2, m_ref, p_row, r);
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[j & 1]);
    }
    if (ok) ok = mbar_wait(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1, status);
    if (ok) {
      tcgen05_fence_after();
      const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
      const bool store = m0 + r < q_len;
      bf16* dst = out + static_cast<size_t>(q_begin + m0 + r) * z.heads * z.vdim + h * z.vdim;
#pragma unroll 1
      for (int c = 0; c < o_cols; c += 32) {
        uint32_t o[32];
        tmem_ld_x32(tmem_o + lane_addr + c, o);
        tmem_ld_wait();
        if (store) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c + i >= z.vdim) continue;              // vdim is a multiple of 8
            uint4 pk;
            pk.x = pack_bf16x2(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv);
            pk.y = pack_bf16x2(__uint_as_float(o[i + 2]) * inv, __uint_as_float(o[i + 3]) * inv);
            pk.z = pack_bf16x2(__uint_as_float(o[i + 4]) * inv, __uint_as_float(o[i + 5]) * inv);
            pk.w = pack_bf16x2(__uint_as_float(o[i + 6]) * inv, __uint_as_float(o[i + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + c + i) = pk;
          }
        }
      }
    }
  }

  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_base, 256);
  }
}

static LatentPrefillSizes latent_prefill_sizes(int heads, int dim, int rot, int vdim, int tok0, int window) {
  return LatentPrefillSizes{heads, dim, rot, vdim, (dim + 63) / 64, (rot + 63) / 64, (vdim + 63) / 64, tok0, window};
}
static int latent_prefill_smem(const LatentPrefillSizes& z) {
  return (z.nb1 + z.nb2) * (kVQBox + kVStages * kVKBox) + kVStages * z.nv * kVKBox + 4 * kVQBox + 256 + 1024;
}

// Columns of one head's packed query row, or 0 when the kernel does not take these sizes (else: latent_attend_any).
extern "C" int forge_latent_prefill_qcols(int dim, int rot, int vdim) {
  if ((dim & 7) || (rot & 7) || (vdim & 7) || dim < 8 || rot < 8 || vdim < 8 || vdim > 128) return 0;
  const LatentPrefillSizes z = latent_prefill_sizes(1, dim, rot, vdim, 0, 0);
  return latent_prefill_smem(z) <= 227 * 1024 ? 64 * (z.nb1 + z.nb2) : 0;
}

extern "C" int forge_make_tmap_2d(CUtensorMap* tm, const void* base, uint64_t rows, uint64_t cols, uint64_t ld,
                                  uint32_t box_rows, int elem_bytes);

// q [tokens - tok0][heads][qcols] (packed); kv [keys][heads * (dim + vdim)]; kr [keys][rot]; sequence s has the step's tokens
// cu_q[s] .. cu_q[s + 1] (its last ones) and the keys cu_k[s] .. cu_k[s + 1] (at least all that they see); out [tokens][heads * vdim].
// Key rows past the last sequence's must hold numbers.
extern "C" int forge_latent_prefill(const void* q, const void* kv, const void* kr, const int* cu_q, const int* cu_k, void* out, int tokens,
                                    int tok0, int keys, int num_seqs, int max_q, int heads, int dim, int rot, int vdim, int window, float scale,
                                    unsigned* status, cudaStream_t stream) {
  if (tokens <= tok0 || num_seqs <= 0) return 0;
  const int qcols = forge_latent_prefill_qcols(dim, rot, vdim);
  if (qcols == 0 || num_seqs > 65535 || heads > 65535) return -1;
  const LatentPrefillSizes z = latent_prefill_sizes(heads, dim, rot, vdim, tok0, window);
  CUtensorMap tm_q, tm_kv, tm_r;
  const uint64_t qw = static_cast<uint64_t>(heads) * qcols, kw = static_cast<uint64_t>(heads) * (dim + vdim);
  if (forge_make_tmap_2d(&tm_q, q, tokens - tok0, qw, qw, kVM, 2) != 0) return -2;
  if (forge_make_tmap_2d(&tm_kv, kv, keys, kw, kw, kVN, 2) != 0) return -2;
  if (forge_make_tmap_2d(&tm_r, kr, keys, rot, rot, kVN, 2) != 0) return -2;
  FORGE_ENSURE_DYN_SMEM(latent_prefill_kernel, 227 * 1024);
  const dim3 grid((max_q + kVM - 1) / kVM, heads, num_seqs);
  return launch_kernel(latent_prefill_kernel, grid, dim3(kVThreads), latent_prefill_smem(z), stream, 0, tm_q, tm_kv, tm_r, cu_q, cu_k,
                       static_cast<bf16*>(out), z, scale * 1.4426950408889634f, status) == cudaSuccess ? 0 : -5;
}

// One warp per key row, 16-byte units.  Of a sequence of lens[s] keys the last cu_k[s + 1] - cu_k[s]; rows past the last sequence's are zero.
__global__ void __launch_bounds__(256) latent_gather_kernel(const bf16* __restrict__ cache, const int* __restrict__ cu_k, const int* __restrict__ lens, int num_seqs,
                                                            const int* __restrict__ block_tables, int table_width, int num_blocks,
                                                            int block_size, int R, int rot, int keys, bf16* __restrict__ c,
                                                            bf16* __restrict__ kr, unsigned* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= keys) return;
  int lo = 0, hi = num_seqs;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (cu_k[mid] <= row) lo = mid; else hi = mid;
  }
  uint4* dc = reinterpret_cast<uint4*>(c + static_cast<size_t>(row) * R);
  uint4* dr = reinterpret_cast<uint4*>(kr + static_cast<size_t>(row) * rot);
  const int uc = R >> 3, ur = rot >> 3;
  if (row >= cu_k[num_seqs]) {
    for (int u = lane; u < uc + ur; u += 32) (u < uc ? dc[u] : dr[u - uc]) = make_uint4(0, 0, 0, 0);
    return;
  }
  const int key = max(lens[lo] - (cu_k[lo + 1] - cu_k[lo]), 0) + row - cu_k[lo];
  int blk = block_tables[static_cast<size_t>(lo) * table_width + min(key / block_size, table_width - 1)];
  if (blk < 0 || blk >= num_blocks) {
    if (lane == 0) set_status(status, kStatusBadIndex);
    blk = 0;
  }
  const uint4* src = reinterpret_cast<const uint4*>(cache + (static_cast<size_t>(blk) * block_size + key % block_size) * (R + rot));
  for (int u = lane; u < uc + ur; u += 32) {
    const uint4 v = src[u];
    if (u < uc) dc[u] = v;
    else dr[u - uc] = v;
  }
}

extern "C" int forge_latent_gather(const void* cache, const int* cu_k, const int* lens, int num_seqs, const int* block_tables, int table_width, int num_blocks,
                                   int block_size, int R, int rot, int keys, void* c, void* kr, unsigned* status, cudaStream_t stream) {
  if (keys <= 0 || num_seqs <= 0) return 0;
  if ((R & 7) || (rot & 7)) return -1;
  return launch_kernel(latent_gather_kernel, dim3((keys + 7) / 8), dim3(256), 0, stream, 0, static_cast<const bf16*>(cache), cu_k, lens, num_seqs,
                       block_tables, table_width, num_blocks, block_size, R, rot, keys, static_cast<bf16*>(c), static_cast<bf16*>(kr),
                       status) == cudaSuccess ? 0 : -2;
}

// q [tokens][heads][dim + rot], tokens ld elements apart -> [tokens][heads][64 (nb1 + nb2)].  A thread moves 8 columns of the unrotated part or 4 pairs.
__global__ void __launch_bounds__(128) latent_pack_q_kernel(const bf16* __restrict__ q, long long ld, bf16* __restrict__ qp, int heads, int dim, int rot,
                                                            int nb1, int nb2, const float* __restrict__ rope, int rope_rows,
                                                            const int* __restrict__ positions) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int pos = positions[t];
  pos = pos < 0 ? 0 : (pos >= rope_rows ? rope_rows - 1 : pos);
  const float* cs = rope + static_cast<size_t>(pos) * rot;
  const int half = rot >> 1, u1 = nb1 * 8, pairs = half >> 2, pad = nb2 * 8 - (rot >> 3), per = u1 + pairs + pad;
  const bf16* src0 = q + static_cast<size_t>(t) * ld;
  bf16* dst0 = qp + static_cast<size_t>(t) * heads * (nb1 + nb2) * 64;
  for (int i = threadIdx.x; i < heads * per; i += blockDim.x) {
    const int h = i / per, u = i % per;
    const bf16* src = src0 + h * (dim + rot);
    bf16* dst = dst0 + static_cast<size_t>(h) * (nb1 + nb2) * 64;
    if (u < u1) {
      *reinterpret_cast<uint4*>(dst + u * 8) = u * 8 < dim ? *reinterpret_cast<const uint4*>(src + u * 8) : make_uint4(0, 0, 0, 0);
    } else if (u < u1 + pairs) {
      const int j = (u - u1) * 4;
      float a[4], b[4];
      load_n<4>(src + dim + j, a);
      load_n<4>(src + dim + half + j, b);
      float x[4], y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        x[e] = a[e] * cs[j + e] - b[e] * cs[half + j + e];
        y[e] = b[e] * cs[j + e] + a[e] * cs[half + j + e];
      }
      store_n<4>(dst + nb1 * 64 + j, x);
      store_n<4>(dst + nb1 * 64 + half + j, y);
    } else {
      *reinterpret_cast<uint4*>(dst + nb1 * 64 + rot + (u - u1 - pairs) * 8) = make_uint4(0, 0, 0, 0);
    }
  }
}

extern "C" int forge_latent_pack_q(const void* q, long long ld, void* qp, int tokens, int heads, int dim, int rot, const float* rope, int rope_rows,
                                   const int* positions, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if ((dim & 7) || (rot & 7) || (ld & 7) || (reinterpret_cast<uintptr_t>(q) & 15)) return -1;
  return launch_kernel(latent_pack_q_kernel, dim3(tokens), dim3(128), 0, stream, 0, static_cast<const bf16*>(q), ld, static_cast<bf16*>(qp), heads,
                       dim, rot, (dim + 63) / 64, (rot + 63) / 64, rope, rope_rows, positions) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
