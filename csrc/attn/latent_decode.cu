// Latent attention of single query tokens on the tensor cores, straight over the paged latents [blocks][block_size][R + rot].
//
// The queries come folded (W_k^T q | rotated part), so all heads of a token share one key row per cached token (its whole
// latent row) and one value row (the first R entries of the SAME row): a tile of keys is read from memory once and serves
// both products for 16 or 32 heads.  CTA = (context chunk, group of 16 kMT heads, sequence), eight warps:
//
//   S = Q K^T    mma.sync m16n8k16, M = 16 heads.  Warp (slice, half) multiplies a quarter of the D columns of Q (held in
//                registers for the whole chunk) with half of the tile's keys; the four partial sums meet in shared memory.
//   softmax      fp32, 16 / kMT threads per head, running maximum and sum in registers.
//   O += P V     every warp owns R / 8 columns.  P is fp32: it enters as bf16 hi + lo halves (two products), so the weights
//                keep 16 mantissa bits.
//
// Key tiles come in by 16-byte cp.async through a ring of two or three stages (the chunk's block ids wait in shared memory); rows are padded to an odd number of 16-byte units, so ldmatrix is
// free of bank conflicts.  Chunks are merged by a second kernel.
#include "../include/launch.cuh"
#include "../include/mma_sync.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kLdThreads = 256, kLdMaxSteps = 9, kLdMaxPairs = 4, kLdMaxChunk = 1024, kLdMaxBlocks = kLdMaxChunk / 16 + 1;

struct LatentDecodeArgs {
  const bf16* qa;            // [seqs][heads][D]
  const bf16* cache;
  const int* block_tables;   // [seqs][table_width]
  const int* lens;           // [seqs] keys visible, the token's own included
  bf16* o;                   // [seqs][heads][R]
  float* part_o;             // [seqs][heads][max_chunks][R]
  float* part_ml;            // [seqs][heads][max_chunks][2]
  int table_width, num_blocks, block_shift, heads, R, D, chunk, max_chunks;
  float scale_log2;
  unsigned* status;
};

__host__ __device__ inline int latent_pitch(int D) { return (D / 8 | 1) * 8; }     // elements; odd number of 16-byte units

template <int kTile, int kMT, int kStages>
__global__ void __launch_bounds__(kLdThreads, kTile == 32 && kMT == 1 ? 2 : 1) latent_decode_kernel(const LatentDecodeArgs p) {
  constexpr int kLdHeads = 16 * kMT, kRowThreads = kLdThreads / kLdHeads, kRowKeys = kTile / kRowThreads;
  constexpr int kSPitch = kTile + 4, kPPitch = kTile + 8;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int pitch = latent_pitch(p.D);
  bf16* sQ = reinterpret_cast<bf16*>(smem_raw);                        // [heads][pitch]
  bf16* sKV = sQ + kLdHeads * pitch;                                   // [kStages][kTile][pitch]
  float* sS = reinterpret_cast<float*>(sKV + kStages * kTile * pitch); // [4][heads][kTile + 4]
  bf16* sP = reinterpret_cast<bf16*>(sS + 4 * kLdHeads * kSPitch);     // [hi, lo][heads][kTile + 8]
  float* sAlpha = reinterpret_cast<float*>(sP + 2 * kLdHeads * kPPitch);       // [heads]
  int* sBlk = reinterpret_cast<int*>(sAlpha + kLdHeads);               // [kLdMaxBlocks]

  pdl_launch_dependents();
  pdl_wait();
  const int ch = blockIdx.x, h0 = blockIdx.y * kLdHeads, seq = blockIdx.z;
  const int len = min(p.lens[seq], p.table_width << p.block_shift);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int k_begin = ch * p.chunk, k_end = min(len, k_begin + p.chunk);
  const int row = threadIdx.x / kRowThreads, sub = threadIdx.x % kRowThreads;   // softmax: head row, lane within its threads
  if (k_begin >= k_end) {
    if (p.max_chunks == 1)                                             // padding of a graph bucket: defined values
      for (int i = threadIdx.x; i < kLdHeads * p.R; i += kLdThreads)
        if (h0 + i / p.R < p.heads) p.o[(static_cast<size_t>(seq) * p.heads + h0) * p.R + i] = __float2bfloat16_rn(0.f);
    return;
  }
  const int units = p.D >> 3;                                          // 16-byte units per row
  const int* table = p.block_tables + static_cast<size_t>(seq) * p.table_width;
  const int blk0 = k_begin >> p.block_shift, n_blk = ((k_end - 1) >> p.block_shift) - blk0 + 1;
  for (int i = threadIdx.x; i < n_blk; i += kLdThreads) {
    int blk = table[blk0 + i];
    if (blk < 0 || blk >= p.num_blocks) {
      set_status(p.status, kStatusBadIndex);
      blk = -1;
    }
    sBlk[i] = blk;
  }
  auto load_tile = [&](int t) {
    bf16* dst = sKV + (t % kStages) * kTile * pitch;
#pragma unroll
    for (int i = 0; i < kTile / 8; ++i) {
      const int r = warp + 8 * i, key = k_begin + t * kTile + r;
      const int blk = key < k_end ? sBlk[(key >> p.block_shift) - blk0] : -1;
      const uint32_t bytes = blk >= 0 ? 16 : 0;
      const bf16* src = p.cache + (blk >= 0 ? ((static_cast<size_t>(blk) << p.block_shift) + (key & ((1 << p.block_shift) - 1))) * p.D : 0);
      const uint32_t to = smem_u32(dst + r * pitch);
      for (int u = lane; u < units; u += 32) cp_async16(to + u * 16, src + u * 8, bytes);
    }
  };
  for (int r = warp; r < kLdHeads; r += kLdThreads / 32) {
    const bool in = h0 + r < p.heads;
    const bf16* src = p.qa + (static_cast<size_t>(seq) * p.heads + (in ? h0 + r : 0)) * p.D;
    for (int u = lane; u < units; u += 32) cp_async16(smem_u32(sQ + r * pitch + u * 8), src + u * 8, in ? 16 : 0);
  }
  __syncthreads();                                                     // block ids
#pragma unroll
  for (int t = 0; t < kStages - 1; ++t) {
    if (k_begin + t * kTile < k_end) load_tile(t);
    cp_async_commit();
  }

  const int slice = warp & 3, half = warp >> 2;
  const int steps = p.D >> 4;
  const int ks0 = slice * steps / 4, ksn = (slice + 1) * steps / 4 - ks0;
  uint32_t qf[kMT][kLdMaxSteps][4];
  float acc[kMT][kLdMaxPairs][2][4];
#pragma unroll
  for (int m = 0; m < kMT; ++m)
#pragma unroll
    for (int i = 0; i < kLdMaxPairs; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) acc[m][i][j][0] = acc[m][i][j][1] = acc[m][i][j][2] = acc[m][i][j][3] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;
  const int pairs = p.R >> 4;
  const int n_tiles = (k_end - k_begin + kTile - 1) / kTile;

  for (int t = 0; t < n_tiles; ++t) {
    cp_async_wait<kStages - 2>();
    __syncthreads();                       // tile t is here; everyone is done with tile t - 1, its stage may be filled again
    if (t + kStages - 1 < n_tiles) load_tile(t + kStages - 1);
    cp_async_commit();
    const uint32_t kv = smem_u32(sKV + (t % kStages) * kTile * pitch);
    if (t == 0) {
#pragma unroll
      for (int m = 0; m < kMT; ++m)
#pragma unroll
        for (int i = 0; i < kLdMaxSteps; ++i)
          if (i < ksn) ldsm_x4(smem_u32(sQ) + ((m * 16 + (lane & 15)) * pitch + (ks0 + i) * 16 + (lane >> 4) * 8) * 2, qf[m][i]);
    }
    {
      constexpr int kNB = kTile / 16;                                  // 8-key blocks per warp
      float s[kMT][kNB][4];
#pragma unroll
      for (int m = 0; m < kMT; ++m)
#pragma unroll
        for (int nb = 0; nb < kNB; ++nb) s[m][nb][0] = s[m][nb][1] = s[m][nb][2] = s[m][nb][3] = 0.f;
#pragma unroll
      for (int i = 0; i < kLdMaxSteps; ++i) {
        if (i < ksn) {
#pragma unroll
          for (int nb = 0; nb < kNB; nb += 2) {
            uint32_t b[4];
            const int r = half * (kTile / 2) + nb * 8 + (lane & 7) + (lane >> 4) * 8;
            ldsm_x4(kv + (r * pitch + (ks0 + i) * 16 + ((lane >> 3) & 1) * 8) * 2, b);
#pragma unroll
            for (int m = 0; m < kMT; ++m) {
              mma16816(s[m][nb], qf[m][i], b[0], b[1]);
              mma16816(s[m][nb + 1], qf[m][i], b[2], b[3]);
            }
          }
        }
      }
      float* dst = sS + slice * kLdHeads * kSPitch + half * (kTile / 2) + 2 * (lane & 3);
#pragma unroll
      for (int m = 0; m < kMT; ++m)
#pragma unroll
        for (int nb = 0; nb < kNB; ++nb) {
          *reinterpret_cast<float2*>(dst + (m * 16 + (lane >> 2)) * kSPitch + nb * 8) = make_float2(s[m][nb][0], s[m][nb][1]);
          *reinterpret_cast<float2*>(dst + (m * 16 + (lane >> 2) + 8) * kSPitch + nb * 8) = make_float2(s[m][nb][2], s[m][nb][3]);
        }
    }
    __syncthreads();
    {
      float s[kRowKeys], mx = -INFINITY;
      const int left = k_end - k_begin - t * kTile;
#pragma unroll
      for (int i = 0; i < kRowKeys; ++i) {
        const int key = sub + kRowThreads * i;
        const float* src = sS + row * kSPitch + key;
        s[i] = key < left ? (src[0] + src[kLdHeads * kSPitch] + src[2 * kLdHeads * kSPitch] + src[3 * kLdHeads * kSPitch]) * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, s[i]);
      }
#pragma unroll
      for (int off = kRowThreads / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_new = fmaxf(m_run, mx);                            // finite: a tile holds at least one visible key
      const float alpha = exp2f(m_run - m_new);
      m_run = m_new;
      l_run *= alpha;
#pragma unroll
      for (int i = 0; i < kRowKeys; ++i) {
        const float w = exp2f(s[i] - m_new);
        l_run += w;
        float hi, lo;
        split_bf16(w, hi, lo);
        sP[row * kPPitch + sub + kRowThreads * i] = __float2bfloat16_rn(hi);
        sP[(kLdHeads + row) * kPPitch + sub + kRowThreads * i] = __float2bfloat16_rn(lo);
      }
      if (sub == 0) sAlpha[row] = alpha;
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < kMT; ++m) {
      const float a0 = sAlpha[m * 16 + (lane >> 2)], a1 = sAlpha[m * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int i = 0; i < kLdMaxPairs; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          acc[m][i][j][0] *= a0;
          acc[m][i][j][1] *= a0;
          acc[m][i][j][2] *= a1;
          acc[m][i][j][3] *= a1;
        }
    }
#pragma unroll
    for (int ks = 0; ks < kTile / 16; ++ks) {
      uint32_t ph[kMT][4], pl[kMT][4];
#pragma unroll
      for (int m = 0; m < kMT; ++m) {
        const uint32_t at = smem_u32(sP) + ((m * 16 + (lane & 15)) * kPPitch + ks * 16 + (lane >> 4) * 8) * 2;
        ldsm_x4(at, ph[m]);
        ldsm_x4(at + kLdHeads * kPPitch * 2, pl[m]);
      }
#pragma unroll
      for (int i = 0; i < kLdMaxPairs; ++i) {
        const int pair = warp + i * 8;
        if (pair < pairs) {
          uint32_t b[4];
          const int r = ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
          ldsm_x4_trans(kv + (r * pitch + pair * 16 + (lane >> 4) * 8) * 2, b);
#pragma unroll
          for (int m = 0; m < kMT; ++m) {
            mma16816(acc[m][i][0], ph[m], b[0], b[1]);
            mma16816(acc[m][i][1], ph[m], b[2], b[3]);
            mma16816(acc[m][i][0], pl[m], b[0], b[1]);
            mma16816(acc[m][i][1], pl[m], b[2], b[3]);
          }
        }
      }
    }
  }
#pragma unroll
  for (int off = kRowThreads / 2; off > 0; off >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, off);
  if (p.max_chunks == 1) {
    __syncthreads();
    if (sub == 0) sAlpha[row] = 1.f / l_run;
    __syncthreads();
  } else if (sub == 0 && h0 + row < p.heads) {
    float* ml = p.part_ml + ((static_cast<size_t>(seq) * p.heads + h0 + row) * p.max_chunks + ch) * 2;
    ml[0] = m_run;
    ml[1] = l_run;
  }
#pragma unroll
  for (int m = 0; m < kMT; ++m)
#pragma unroll
    for (int i = 0; i < kLdMaxPairs; ++i) {
      const int pair = warp + i * 8;
      if (pair >= pairs) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = m * 16 + (lane >> 2) + e * 8, c = pair * 16 + j * 8 + 2 * (lane & 3);
          if (h0 + r >= p.heads) continue;
          const float v0 = acc[m][i][j][2 * e], v1 = acc[m][i][j][2 * e + 1];
          const size_t hr = static_cast<size_t>(seq) * p.heads + h0 + r;
          if (p.max_chunks == 1)
            *reinterpret_cast<uint32_t*>(p.o + hr * p.R + c) = pack_bf16x2(v0 * sAlpha[r], v1 * sAlpha[r]);
          else
            *reinterpret_cast<float2*>(p.part_o + (hr * p.max_chunks + ch) * p.R + c) = make_float2(v0, v1);
        }
    }
}

// One CTA per (head, sequence): the chunks' partial sums, weighted by their maxima.
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                           const int* __restrict__ lens, bf16* __restrict__ o, int heads, int R, int chunk,
                                                           int max_chunks, int max_len) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, seq = blockIdx.y;
  const size_t hr = static_cast<size_t>(seq) * heads + h;
  const int len = min(lens[seq], max_len);
  const int n = len > 0 ? min((len + chunk - 1) / chunk, max_chunks) : 0;
  const float* ml = part_ml + hr * max_chunks * 2;
  float m = -INFINITY;
  for (int c = 0; c < n; ++c) m = fmaxf(m, ml[2 * c]);
  float l = 0.f;
  for (int c = 0; c < n; ++c) l += ml[2 * c + 1] * exp2f(ml[2 * c] - m);
  const float inv = n > 0 ? 1.f / l : 0.f;
  for (int i = threadIdx.x * 4; i < R; i += blockDim.x * 4) {
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c = 0; c < n; ++c) {
      const float w = exp2f(ml[2 * c] - m) * inv;
      const float4 v = *reinterpret_cast<const float4*>(part_o + (hr * max_chunks + c) * R + i);
      s.x = fmaf(w, v.x, s.x);
      s.y = fmaf(w, v.y, s.y);
      s.z = fmaf(w, v.z, s.z);
      s.w = fmaf(w, v.w, s.w);
    }
    *reinterpret_cast<uint2*>(o + hr * R + i) = make_uint2(pack_bf16x2(s.x, s.y), pack_bf16x2(s.z, s.w));
  }
}

template <int kTile, int kMT, int kStages>
static int launch_latent_decode(const LatentDecodeArgs& p, int seqs, cudaStream_t stream) {
  constexpr int kHeads = 16 * kMT;
  auto smem = [](int D) {
    return static_cast<int>((kHeads + kStages * kTile) * latent_pitch(D) * 2 + 4 * kHeads * (kTile + 4) * 4 + 2 * kHeads * (kTile + 8) * 2 +
                            kHeads * 4 + kLdMaxBlocks * 4);
  };
  auto kern = latent_decode_kernel<kTile, kMT, kStages>;
  FORGE_ENSURE_DYN_SMEM(kern, smem(64 * kLdMaxSteps));
  return launch_kernel(kern, dim3(p.max_chunks, (p.heads + kHeads - 1) / kHeads, seqs), dim3(kLdThreads), smem(p.D), stream, 0, p) == cudaSuccess ? 0 : -2;
}

// 1 if the kernel takes these sizes (else: latent_attend_any).
extern "C" int forge_latent_decode_ok(int R, int rot, int block_size) {
  return R % 16 == 0 && rot % 16 == 0 && R >= 16 && R <= 16 * 8 * kLdMaxPairs && R + rot <= 64 * kLdMaxSteps && block_size >= 16 && (block_size & (block_size - 1)) == 0;
}

// qa [seqs][heads][R + rot] bf16; lens = keys visible per sequence; part_* needed when max_chunks > 1.
extern "C" int forge_latent_decode(const void* qa, const void* cache, const int* block_tables, const int* lens, void* o, float* part_o,
                                   float* part_ml, int seqs, int heads, int R, int rot, int table_width, int num_blocks, int block_size,
                                   int chunk, int max_chunks, int tile, float scale, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (!forge_latent_decode_ok(R, rot, block_size) || chunk < 64 || chunk % 64 || chunk > kLdMaxChunk || (tile != 32 && tile != 64) || seqs > 65535 ||
      (reinterpret_cast<uintptr_t>(qa) & 15) || (reinterpret_cast<uintptr_t>(cache) & 15))
    return -1;
  int shift = 0;
  while ((1 << shift) < block_size) ++shift;
  const LatentDecodeArgs p = {static_cast<const bf16*>(qa), static_cast<const bf16*>(cache), block_tables, lens, static_cast<bf16*>(o), part_o,
                              part_ml, table_width, num_blocks, shift, heads, R, R + rot, chunk, max_chunks, scale * 1.4426950408889634f, status};
  const int rc = heads > 16 ? launch_latent_decode<32, 2, 3>(p, seqs, stream)
                 : tile == 32 ? launch_latent_decode<32, 1, 2>(p, seqs, stream) : launch_latent_decode<64, 1, 2>(p, seqs, stream);
  if (rc != 0) return rc;
  if (max_chunks == 1) return 0;
  return launch_kernel(latent_merge_kernel, dim3(heads, seqs), dim3(128), 0, stream, 0, part_o, part_ml, lens, static_cast<bf16*>(o), heads, R,
                       chunk, max_chunks, table_width * block_size) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
