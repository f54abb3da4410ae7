// Latent attention of single query tokens on the tensor cores, straight over the paged latents [blocks][block_size][R + rot].
//
// The queries come folded (W_k^T q | rotated part), so all heads of a token share one key row per cached token (its whole
// latent row) and one value row (the first R entries of the SAME row): a tile of keys is read from memory once and serves
// both products for 16 heads.  CTA = (context chunk, group of 16 heads, sequence), eight warps:
//
//   S = Q K^T    mma.sync m16n8k16, M = the 16 heads.  Warp (slice, half) multiplies a quarter of the D columns of Q (held in
//                registers for the whole chunk) with half of the tile's keys; the four partial sums meet in shared memory.
//   softmax      fp32, 16 threads per head, running maximum and sum in registers.
//   O += P V     every warp owns R / 8 columns.  P is fp32: it enters as bf16 hi + lo halves (two products), so the weights
//                keep 16 mantissa bits.
//
// Key tiles come in by 16-byte cp.async, double-buffered; rows are padded to an odd number of 16-byte units, so ldmatrix is
// free of bank conflicts.  Chunks are merged by a second kernel.
#include "../include/launch.cuh"
#include "../include/mma_sync.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kLdThreads = 256, kLdHeads = 16, kLdMaxSteps = 9, kLdMaxPairs = 4;

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

template <int kTile>
__global__ void __launch_bounds__(kLdThreads, kTile == 32 ? 2 : 1) latent_decode_kernel(const LatentDecodeArgs p) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int pitch = latent_pitch(p.D);
  bf16* sQ = reinterpret_cast<bf16*>(smem_raw);                        // [16][pitch]
  bf16* sKV = sQ + kLdHeads * pitch;                                   // [2][kTile][pitch]
  float* sS = reinterpret_cast<float*>(sKV + 2 * kTile * pitch);       // [4][16][kTile + 4]
  bf16* sP = reinterpret_cast<bf16*>(sS + 4 * kLdHeads * (kTile + 4)); // [2][16][kTile + 8]
  float* sAlpha = reinterpret_cast<float*>(sP + 2 * kLdHeads * (kTile + 8));   // [16]
  constexpr int kSPitch = kTile + 4, kPPitch = kTile + 8;

  pdl_launch_dependents();
  pdl_wait();
  const int ch = blockIdx.x, h0 = blockIdx.y * kLdHeads, seq = blockIdx.z;
  const int len = min(p.lens[seq], p.table_width << p.block_shift);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int k_begin = ch * p.chunk, k_end = min(len, k_begin + p.chunk);
  const int row = threadIdx.x >> 4, sub = threadIdx.x & 15;            // softmax: head row, lane within its 16 threads
  if (k_begin >= k_end) {
    if (p.max_chunks == 1)                                             // padding of a graph bucket: defined values
      for (int i = threadIdx.x; i < kLdHeads * p.R; i += kLdThreads)
        if (h0 + i / p.R < p.heads) p.o[(static_cast<size_t>(seq) * p.heads + h0) * p.R + i] = __float2bfloat16_rn(0.f);
    return;
  }
  const int units = p.D >> 3;                                          // 16-byte units per row
  const int* table = p.block_tables + static_cast<size_t>(seq) * p.table_width;
  auto load_tile = [&](int t) {
    bf16* dst = sKV + (t & 1) * kTile * pitch;
    for (int r = warp; r < kTile; r += kLdThreads / 32) {
      const int key = k_begin + t * kTile + r;
      const bf16* src = p.cache;
      uint32_t bytes = 0;
      if (key < k_end) {
        const int blk = table[key >> p.block_shift];
        if (blk >= 0 && blk < p.num_blocks) {
          src = p.cache + ((static_cast<size_t>(blk) << p.block_shift) + (key & ((1 << p.block_shift) - 1))) * p.D;
          bytes = 16;
        } else if (lane == 0) {
          set_status(p.status, kStatusBadIndex);
        }
      }
      for (int u = lane; u < units; u += 32) cp_async16(smem_u32(dst + r * pitch + u * 8), bytes ? src + u * 8 : src, bytes);
    }
  };
  for (int r = warp; r < kLdHeads; r += kLdThreads / 32) {
    const bool in = h0 + r < p.heads;
    const bf16* src = p.qa + (static_cast<size_t>(seq) * p.heads + (in ? h0 + r : 0)) * p.D;
    for (int u = lane; u < units; u += 32) cp_async16(smem_u32(sQ + r * pitch + u * 8), src + u * 8, in ? 16 : 0);
  }
  load_tile(0);
  cp_async_commit();

  const int slice = warp & 3, half = warp >> 2;
  const int steps = p.D >> 4;
  const int ks0 = slice * steps / 4, ksn = (slice + 1) * steps / 4 - ks0;
  uint32_t qf[kLdMaxSteps][4];
  float acc[kLdMaxPairs][2][4];
#pragma unroll
  for (int i = 0; i < kLdMaxPairs; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;
  const int pairs = p.R >> 4;
  const int n_tiles = (k_end - k_begin + kTile - 1) / kTile;

  for (int t = 0; t < n_tiles; ++t) {
    if (t + 1 < n_tiles) load_tile(t + 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t kv = smem_u32(sKV + (t & 1) * kTile * pitch);
    if (t == 0) {
#pragma unroll
      for (int i = 0; i < kLdMaxSteps; ++i)
        if (i < ksn) ldsm_x4(smem_u32(sQ) + ((lane & 15) * pitch + (ks0 + i) * 16 + (lane >> 4) * 8) * 2, qf[i]);
    }
    {
      constexpr int kNB = kTile / 16;                                  // 8-key blocks per warp
      float s[kNB][4];
#pragma unroll
      for (int nb = 0; nb < kNB; ++nb) s[nb][0] = s[nb][1] = s[nb][2] = s[nb][3] = 0.f;
#pragma unroll
      for (int i = 0; i < kLdMaxSteps; ++i) {
        if (i < ksn) {
#pragma unroll
          for (int nb = 0; nb < kNB; nb += 2) {
            uint32_t b[4];
            const int r = half * (kTile / 2) + nb * 8 + (lane & 7) + (lane >> 4) * 8;
            ldsm_x4(kv + (r * pitch + (ks0 + i) * 16 + ((lane >> 3) & 1) * 8) * 2, b);
            mma16816(s[nb], qf[i], b[0], b[1]);
            mma16816(s[nb + 1], qf[i], b[2], b[3]);
          }
        }
      }
      float* dst = sS + slice * kLdHeads * kSPitch + half * (kTile / 2) + 2 * (lane & 3);
#pragma unroll
      for (int nb = 0; nb < kNB; ++nb) {
        *reinterpret_cast<float2*>(dst + (lane >> 2) * kSPitch + nb * 8) = make_float2(s[nb][0], s[nb][1]);
        *reinterpret_cast<float2*>(dst + ((lane >> 2) + 8) * kSPitch + nb * 8) = make_float2(s[nb][2], s[nb][3]);
      }
    }
    __syncthreads();
    {
      float s[kTile / 16], mx = -INFINITY;
      const int left = k_end - k_begin - t * kTile;
#pragma unroll
      for (int i = 0; i < kTile / 16; ++i) {
        const int key = sub + 16 * i;
        const float* src = sS + row * kSPitch + key;
        s[i] = key < left ? (src[0] + src[kLdHeads * kSPitch] + src[2 * kLdHeads * kSPitch] + src[3 * kLdHeads * kSPitch]) * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, s[i]);
      }
#pragma unroll
      for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_new = fmaxf(m_run, mx);                            // finite: a tile holds at least one visible key
      const float alpha = exp2f(m_run - m_new);
      m_run = m_new;
      l_run *= alpha;
#pragma unroll
      for (int i = 0; i < kTile / 16; ++i) {
        const float w = exp2f(s[i] - m_new);
        l_run += w;
        float hi, lo;
        split_bf16(w, hi, lo);
        sP[row * kPPitch + sub + 16 * i] = __float2bfloat16_rn(hi);
        sP[(kLdHeads + row) * kPPitch + sub + 16 * i] = __float2bfloat16_rn(lo);
      }
      if (sub == 0) sAlpha[row] = alpha;
    }
    __syncthreads();
    {
      const float a0 = sAlpha[lane >> 2], a1 = sAlpha[(lane >> 2) + 8];
      uint32_t ph[kTile / 16][4], pl[kTile / 16][4];
#pragma unroll
      for (int ks = 0; ks < kTile / 16; ++ks) {
        const uint32_t at = smem_u32(sP) + ((lane & 15) * kPPitch + ks * 16 + (lane >> 4) * 8) * 2;
        ldsm_x4(at, ph[ks]);
        ldsm_x4(at + kLdHeads * kPPitch * 2, pl[ks]);
      }
#pragma unroll
      for (int i = 0; i < kLdMaxPairs; ++i) {
        const int pair = warp + i * 8;
        if (pair < pairs) {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            acc[i][j][0] *= a0;
            acc[i][j][1] *= a0;
            acc[i][j][2] *= a1;
            acc[i][j][3] *= a1;
          }
#pragma unroll
          for (int ks = 0; ks < kTile / 16; ++ks) {
            uint32_t b[4];
            const int r = ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
            ldsm_x4_trans(kv + (r * pitch + pair * 16 + (lane >> 4) * 8) * 2, b);
            mma16816(acc[i][0], ph[ks], b[0], b[1]);
            mma16816(acc[i][1], ph[ks], b[2], b[3]);
            mma16816(acc[i][0], pl[ks], b[0], b[1]);
            mma16816(acc[i][1], pl[ks], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();                                                   // the tile, S and P may be overwritten
  }
#pragma unroll
  for (int off = 8; off > 0; off >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, off);
  if (p.max_chunks == 1) {
    if (sub == 0) sAlpha[row] = 1.f / l_run;
    __syncthreads();
  } else if (sub == 0 && h0 + row < p.heads) {
    float* ml = p.part_ml + ((static_cast<size_t>(seq) * p.heads + h0 + row) * p.max_chunks + ch) * 2;
    ml[0] = m_run;
    ml[1] = l_run;
  }
#pragma unroll
  for (int i = 0; i < kLdMaxPairs; ++i) {
    const int pair = warp + i * 8;
    if (pair >= pairs) continue;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = (lane >> 2) + e * 8, c = pair * 16 + j * 8 + 2 * (lane & 3);
        if (h0 + r >= p.heads) continue;
        const float v0 = acc[i][j][2 * e], v1 = acc[i][j][2 * e + 1];
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

static size_t latent_decode_smem(int D, int tile) {
  return static_cast<size_t>(kLdHeads + 2 * tile) * latent_pitch(D) * 2 + 4 * kLdHeads * (tile + 4) * 4 + 2 * kLdHeads * (tile + 8) * 2 + kLdHeads * 4;
}

// 1 if the kernel takes these sizes (else: latent_attend_any).
extern "C" int forge_latent_decode_ok(int R, int rot, int block_size) {
  return R % 16 == 0 && rot % 16 == 0 && R >= 16 && R <= 16 * 8 * kLdMaxPairs && R + rot <= 64 * kLdMaxSteps && (block_size & (block_size - 1)) == 0;
}

// qa [seqs][heads][R + rot] bf16; lens = keys visible per sequence; part_* needed when max_chunks > 1.
extern "C" int forge_latent_decode(const void* qa, const void* cache, const int* block_tables, const int* lens, void* o, float* part_o,
                                   float* part_ml, int seqs, int heads, int R, int rot, int table_width, int num_blocks, int block_size,
                                   int chunk, int max_chunks, int tile, float scale, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (!forge_latent_decode_ok(R, rot, block_size) || chunk < 1 || chunk % tile || (tile != 32 && tile != 64) || seqs > 65535 ||
      (reinterpret_cast<uintptr_t>(qa) & 15) || (reinterpret_cast<uintptr_t>(cache) & 15))
    return -1;
  int shift = 0;
  while ((1 << shift) < block_size) ++shift;
  const LatentDecodeArgs p = {static_cast<const bf16*>(qa), static_cast<const bf16*>(cache), block_tables, lens, static_cast<bf16*>(o), part_o,
                              part_ml, table_width, num_blocks, shift, heads, R, R + rot, chunk, max_chunks, scale * 1.4426950408889634f, status};
  const dim3 grid(max_chunks, (heads + kLdHeads - 1) / kLdHeads, seqs);
  const size_t smem = latent_decode_smem(R + rot, tile);
  if (tile == 32) {
    FORGE_ENSURE_DYN_SMEM(latent_decode_kernel<32>, static_cast<int>(latent_decode_smem(64 * kLdMaxSteps, 32)));
    if (launch_kernel(latent_decode_kernel<32>, grid, dim3(kLdThreads), smem, stream, 0, p) != cudaSuccess) return -2;
  } else {
    FORGE_ENSURE_DYN_SMEM(latent_decode_kernel<64>, static_cast<int>(latent_decode_smem(64 * kLdMaxSteps, 64)));
    if (launch_kernel(latent_decode_kernel<64>, grid, dim3(kLdThreads), smem, stream, 0, p) != cudaSuccess) return -2;
  }
  if (max_chunks == 1) return 0;
  return launch_kernel(latent_merge_kernel, dim3(heads, seqs), dim3(128), 0, stream, 0, part_o, part_ml, lens, static_cast<bf16*>(o), heads, R,
                       chunk, max_chunks, table_width * block_size) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
