// Mixture of experts: routing and the shuffling of rows.
//
//   router          logits (fp32) -> sigmoid -> the `top` largest scores of a token (ties: the lower expert)
//   moe_plan        (token, choice) -> row of the expert-sorted buffer; every expert's rows start on a multiple of `tile`, so
//                   a tile of rows has one expert (tile_expert; -1 past the last tile in use)
//   moe_scatter     row = score * token, the score in fp32: it multiplies the expert's INPUT
//
// Rows between an expert's last token and its next tile boundary are never written nor read back.
#include "../include/launch.cuh"
#include "../include/mma_sync.cuh"
#include "../include/scalar.cuh"

namespace forge {

// The `top` largest of a token's scores, by one warp; the scores in shared memory are used up.
__device__ __forceinline__ void choose_top(float* score, int E, int top, int lane, int* experts, float* weights) {
  for (int j = 0; j < top; ++j) {
    float best = -1.f;
    int at = E;
    for (int e = lane; e < E; e += 32)
      if (score[e] > best) { best = score[e]; at = e; }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
      const float v = __shfl_xor_sync(0xffffffffu, best, off);
      const int i = __shfl_xor_sync(0xffffffffu, at, off);
      if (v > best || (v == best && i < at)) { best = v; at = i; }
    }
    if (at >= E) at = 0;                          // only if every score is NaN
    if (lane == 0) {
      experts[j] = at;
      weights[j] = best;
      score[at] = -2.f;
    }
    __syncwarp();
  }
}

// bf16, W a multiple of 32, E <= 256: CTA = 16 MT tokens, the eight warps split W.  The order of the columns in a dot product is
// free, so a lane loads eight consecutive columns of its row (16 bytes) and uses them as the four column pairs of two mma
// k-steps, for tokens and experts alike: no shared memory on the way in.  The warps' partial logits are added in a fixed order.
template <int MT>
__global__ void __launch_bounds__(256) router_mma_kernel(const bf16* __restrict__ h, const bf16* __restrict__ w, int T, int W, int E, int top,
                                                         int* __restrict__ experts, float* __restrict__ weights) {
  extern __shared__ float sm_part[];               // [8][16 MT][Ep]
  constexpr int kTok = 16 * MT, kGroup = 8;        // 8-expert blocks per pass
  const int Ep = (E + 7) & ~7;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int t0 = blockIdx.x * kTok;
  pdl_launch_dependents();
  pdl_wait();
  for (int e0 = 0; e0 < E; e0 += 8 * kGroup) {
    float acc[MT][kGroup][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < kGroup; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
    for (int c = warp * 32; c < W; c += 256) {
      uint4 a[MT][2];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = t0 + m * 16 + r * 8 + g;
          a[m][r] = t < T ? *reinterpret_cast<const uint4*>(h + static_cast<size_t>(t) * W + c + q * 8) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
      for (int n = 0; n < kGroup; ++n) {
        const int e = e0 + n * 8 + g;
        if (e0 + n * 8 >= E) continue;
        const uint4 b = e < E ? *reinterpret_cast<const uint4*>(w + static_cast<size_t>(e) * W + c + q * 8) : make_uint4(0, 0, 0, 0);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          const uint32_t lo[4] = {a[m][0].x, a[m][1].x, a[m][0].y, a[m][1].y}, hi[4] = {a[m][0].z, a[m][1].z, a[m][0].w, a[m][1].w};
          mma16816(acc[m][n], lo, b.x, b.y);
          mma16816(acc[m][n], hi, b.z, b.w);
        }
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < kGroup; ++n) {
        if (e0 + n * 8 >= E) continue;
        float* dst = sm_part + (static_cast<size_t>(warp) * kTok + m * 16 + g) * Ep + e0 + n * 8 + 2 * q;
        *reinterpret_cast<float2*>(dst) = make_float2(acc[m][n][0], acc[m][n][1]);
        *reinterpret_cast<float2*>(dst + 8 * Ep) = make_float2(acc[m][n][2], acc[m][n][3]);
      }
  }
  __syncthreads();
  for (int t = warp; t < kTok && t0 + t < T; t += 8) {
    float* score = sm_part + static_cast<size_t>(t) * Ep;
    for (int e = lane; e < E; e += 32) {
      float z = score[e];
#pragma unroll
      for (int k = 1; k < 8; ++k) z += score[static_cast<size_t>(k) * kTok * Ep + e];
      score[e] = 1.f / (1.f + expf(-z));
    }
    __syncwarp();
    choose_top(score, E, top, lane, experts + static_cast<size_t>(t0 + t) * top, weights + static_cast<size_t>(t0 + t) * top);
  }
}

// The same for many tokens and at most 64 experts: CTA = 128 tokens, a warp owns 16 of them over the whole width; the router matrix
// passes through shared memory, 128 columns at a time, so it is read once per 128 tokens.  A token's scores end up in the four
// lanes of its row, which choose the experts among themselves.
constexpr int kRtCols = 128, kRtPitch = kRtCols + 32;       // a row stride of 4 (mod 8) 16-byte units: conflict-free 16-byte reads

template <int NB>
__global__ void __launch_bounds__(256) router_tall_kernel(const bf16* __restrict__ h, const bf16* __restrict__ w, int T, int W, int E, int top,
                                                          int* __restrict__ experts, float* __restrict__ weights) {
  __shared__ __align__(16) bf16 sw[2][NB * 8][kRtPitch];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int t0 = blockIdx.x * 128 + warp * 16;
  auto load_w = [&](int c0, int st) {
    for (int i = threadIdx.x; i < NB * 8 * (kRtCols / 8); i += 256) {
      const int e = i / (kRtCols / 8), u = i % (kRtCols / 8);
      const bool in = e < E && c0 + u * 8 < W;
      cp_async16(smem_u32(&sw[st][e][u * 8]), in ? w + static_cast<size_t>(e) * W + c0 + u * 8 : w, in ? 16 : 0);
    }
    cp_async_commit();
  };
  pdl_launch_dependents();
  load_w(0, 0);                                     // weights do not depend on the kernel before
  pdl_wait();
  const bf16* rows[2] = {h + static_cast<size_t>(min(t0 + g, T - 1)) * W + q * 8, h + static_cast<size_t>(min(t0 + 8 + g, T - 1)) * W + q * 8};
  uint4 next[4][2];                                 // the tokens' columns of the next 128
  auto load_h = [&](int c0) {
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r) next[i][r] = c0 + i * 32 < W ? *reinterpret_cast<const uint4*>(rows[r] + c0 + i * 32) : make_uint4(0, 0, 0, 0);
  };
  load_h(0);
  float acc[NB][4];
#pragma unroll
  for (int n = 0; n < NB; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
  int st = 0;
  for (int c0 = 0; c0 < W; c0 += kRtCols, st ^= 1) {
    cp_async_wait<0>();
    __syncthreads();                                // the columns are here; everyone is done with the other stage
    if (c0 + kRtCols < W) load_w(c0 + kRtCols, st ^ 1);
    uint4 a[4][2];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r) a[i][r] = next[i][r];
    if (c0 + kRtCols < W) load_h(c0 + kRtCols);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const uint32_t lo[4] = {a[i][0].x, a[i][1].x, a[i][0].y, a[i][1].y}, hi[4] = {a[i][0].z, a[i][1].z, a[i][0].w, a[i][1].w};
#pragma unroll
      for (int n = 0; n < NB; ++n) {
        const uint4 b = *reinterpret_cast<const uint4*>(&sw[st][n * 8 + g][i * 32 + q * 8]);
        mma16816(acc[n], lo, b.x, b.y);
        mma16816(acc[n], hi, b.z, b.w);
      }
    }
  }
  // lane (g, q) holds the logits of tokens g and g + 8 for experts 8 n + 2 q, + 1
#pragma unroll
  for (int n = 0; n < NB; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = n * 8 + 2 * q + (e & 1) < E ? 1.f / (1.f + expf(-acc[n][e])) : -2.f;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = t0 + r * 8 + g;
    for (int j = 0; j < top; ++j) {
      float best = -1.f;
      int at = E;
#pragma unroll
      for (int n = 0; n < NB; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          if (acc[n][2 * r + e] > best) { best = acc[n][2 * r + e]; at = n * 8 + 2 * q + e; }
#pragma unroll
      for (int off = 1; off < 4; off <<= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, best, off);
        const int i = __shfl_xor_sync(0xffffffffu, at, off);
        if (v > best || (v == best && i < at)) { best = v; at = i; }
      }
      if (at >= E) at = 0;                          // only if every score is NaN
#pragma unroll
      for (int n = 0; n < NB; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          if (n * 8 + 2 * q + e == at) acc[n][2 * r + e] = -2.f;
      if (q == 0 && t < T) {
        experts[static_cast<size_t>(t) * top + j] = at;
        weights[static_cast<size_t>(t) * top + j] = best;
      }
    }
  }
}

// CTA = one token; one warp per expert at a time.
template <typename T, int N>
__global__ void __launch_bounds__(256) router_kernel(const T* __restrict__ h, const T* __restrict__ w, int W, int E, int top,
                                                     int* __restrict__ experts, float* __restrict__ weights) {
  extern __shared__ float score[];
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* row = h + t * W;
  for (int e = warp; e < E; e += blockDim.x >> 5) {
    const T* we = w + static_cast<size_t>(e) * W;
    float z = 0.f;
    for (int i = lane * N; i < W; i += 32 * N) {
      float a[N], b[N];
      load_n<N>(row + i, a);
      load_n<N>(we + i, b);
#pragma unroll
      for (int q = 0; q < N; ++q) z = fmaf(a[q], b[q], z);
    }
    z = warp_sum_f(z);
    if (lane == 0) score[e] = 1.f / (1.f + expf(-z));
  }
  __syncthreads();
  if (warp == 0) choose_top(score, E, top, lane, experts + t * top, weights + t * top);
}

extern "C" int forge_router(int fp32, const void* h, const void* w, int T_, int W, int E, int top, int* experts, float* weights,
                            cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (E > 4096 || top < 1 || top > E) return -1;
  const bool v4 = (W & 3) == 0;
  const size_t smem = static_cast<size_t>(E) * 4;
  if (fp32) {
    auto k = v4 ? router_kernel<float, 4> : router_kernel<float, 1>;
    return launch_kernel(k, dim3(T_), dim3(256), smem, stream, 0, static_cast<const float*>(h), static_cast<const float*>(w), W, E, top, experts, weights) == cudaSuccess ? 0 : -2;
  }
  if (W % 32 == 0 && E <= 256 && (reinterpret_cast<uintptr_t>(h) & 15) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0) {
    if (T_ >= 1024 && E <= 64) {
      auto k = E <= 16 ? router_tall_kernel<2> : E <= 32 ? router_tall_kernel<4> : router_tall_kernel<8>;
      return launch_kernel(k, dim3((T_ + 127) / 128), dim3(256), 0, stream, 0, static_cast<const bf16*>(h), static_cast<const bf16*>(w), T_, W, E, top, experts, weights) == cudaSuccess ? 0 : -2;
    }
    const int Ep = (E + 7) & ~7;
    const bool two = T_ > 2048 && E <= 128;        // more tokens per CTA halve the reads of the router matrix
    const dim3 grid((T_ + (two ? 31 : 15)) / (two ? 32 : 16));
    const size_t part = static_cast<size_t>(8) * (two ? 32 : 16) * Ep * 4;
    if (two) {
      FORGE_ENSURE_DYN_SMEM(router_mma_kernel<2>, 8 * 32 * 128 * 4);
      return launch_kernel(router_mma_kernel<2>, grid, dim3(256), part, stream, 0, static_cast<const bf16*>(h), static_cast<const bf16*>(w), T_, W, E, top, experts, weights) == cudaSuccess ? 0 : -2;
    }
    FORGE_ENSURE_DYN_SMEM(router_mma_kernel<1>, 8 * 16 * 256 * 4);
    return launch_kernel(router_mma_kernel<1>, grid, dim3(256), part, stream, 0, static_cast<const bf16*>(h), static_cast<const bf16*>(w), T_, W, E, top, experts, weights) == cudaSuccess ? 0 : -2;
  }
  auto k = v4 ? router_kernel<bf16, 4> : router_kernel<bf16, 1>;
  return launch_kernel(k, dim3(T_), dim3(256), smem, stream, 0, static_cast<const bf16*>(h), static_cast<const bf16*>(w), W, E, top, experts, weights) == cudaSuccess ? 0 : -2;
}

constexpr int kPlanThreads = 1024;

// One CTA.  smem: counts [E], next row [E].
__global__ void __launch_bounds__(kPlanThreads) moe_plan_kernel(const int* __restrict__ experts, int n, int E, int tile, int max_tiles,
                                                                int* __restrict__ pos, int* __restrict__ tile_expert,
                                                                int* __restrict__ num_tiles, unsigned* status) {
  extern __shared__ int sm_plan[];
  int* count = sm_plan;
  int* next = sm_plan + E;
  pdl_launch_dependents();
  pdl_wait();
  for (int e = threadIdx.x; e < E; e += kPlanThreads) count[e] = 0;
  __syncthreads();
  auto expert_of = [&](int i) {                   // an index out of range is reported and becomes expert 0
    const int e = experts[i];
    if (e >= 0 && e < E) return e;
    set_status(status, kStatusBadIndex);
    return 0;
  };
  for (int i = threadIdx.x; i < n; i += kPlanThreads) atomicAdd(&count[expert_of(i)], 1);
  __syncthreads();
  if (threadIdx.x < 32) {                         // running sum of tiles, 32 experts at a time
    int base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int tiles = e < E ? (count[e] + tile - 1) / tile : 0;
      int incl = tiles;
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, incl, off);
        if (threadIdx.x >= off) incl += v;
      }
      if (e < E) next[e] = (base + incl - tiles) * tile;
      base += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (threadIdx.x == 0) num_tiles[0] = base;
  }
  for (int i = threadIdx.x; i < max_tiles; i += kPlanThreads) tile_expert[i] = -1;
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += kPlanThreads)
    for (int k = 0; k < (count[e] + tile - 1) / tile && next[e] / tile + k < max_tiles; ++k) tile_expert[next[e] / tile + k] = e;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += kPlanThreads) pos[i] = atomicAdd(&next[expert_of(i)], 1);
}

// max_tiles >= n / tile + E rounded up: the caller's buffer has max_tiles * tile rows.
extern "C" int forge_moe_plan(const int* experts, int n, int E, int tile, int max_tiles, int* pos, int* tile_expert, int* num_tiles,
                              unsigned* status, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (E > 4096 || tile < 1) return -1;
  return launch_kernel(moe_plan_kernel, dim3(1), dim3(kPlanThreads), static_cast<size_t>(E) * 8, stream, 0, experts, n, E, tile, max_tiles,
                       pos, tile_expert, num_tiles, status) == cudaSuccess ? 0 : -2;
}

template <typename T, int N>
__global__ void __launch_bounds__(256) moe_scatter_kernel(const T* __restrict__ h, const int* __restrict__ pos,
                                                          const float* __restrict__ weights, int top, int W, T* __restrict__ xs,
                                                          int xs_rows, unsigned* status) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  for (int c = threadIdx.x * N; c < W; c += blockDim.x * N) {
    float v[N];
    load_n<N>(h + t * W + c, v);
    for (int j = 0; j < top; ++j) {
      const float s = weights[t * top + j];
      const int row = pos[t * top + j];
      if (row < 0 || row >= xs_rows) {
        set_status(status, kStatusBadIndex);
        continue;
      }
      float x[N];
#pragma unroll
      for (int e = 0; e < N; ++e) x[e] = s * v[e];
      store_n<N>(xs + static_cast<size_t>(row) * W + c, x);
    }
  }
}

extern "C" int forge_moe_scatter(int fp32, const void* h, const int* pos, const float* weights, int n, int top, int W, void* xs, int xs_rows,
                                 unsigned* status, cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v4 = (W & 3) == 0;
  if (fp32) {
    auto k = v4 ? moe_scatter_kernel<float, 4> : moe_scatter_kernel<float, 1>;
    return launch_kernel(k, dim3(n / top), dim3(256), 0, stream, 0, static_cast<const float*>(h), pos, weights, top, W, static_cast<float*>(xs), xs_rows, status) == cudaSuccess ? 0 : -2;
  }
  auto k = v4 ? moe_scatter_kernel<bf16, 4> : moe_scatter_kernel<bf16, 1>;
  return launch_kernel(k, dim3(n / top), dim3(256), 0, stream, 0, static_cast<const bf16*>(h), pos, weights, top, W, static_cast<bf16*>(xs), xs_rows, status) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
