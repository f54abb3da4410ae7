// Mixture of experts: routing and the shuffling of rows.
//
//   router          logits (fp32) -> the `top` largest of a token (ties: the lower expert), weighted by the sigmoid of each or
//                   by the softmax over the chosen ones.  With sigmoids the choice may go by score + correction, and be limited to
//                   the experts of the `keep` groups of neighbours whose two best experts are best together
//   moe_plan        (token, choice) -> row of the expert-sorted buffer; every expert's rows start on a multiple of `tile`, so
//                   a tile of rows has one expert (tile_expert; -1 past the last tile in use)
//   moe_scatter     row = token, or weight * token (weight in fp32) where the weight multiplies the expert's INPUT
//
// Rows between an expert's last token and its next tile boundary are never written nor read back.
#include "../include/launch.cuh"
#include "../include/mma_sync.cuh"
#include "../include/scalar.cuh"

namespace forge {

// The `top` largest of a token's scores, by one warp; the scores in shared memory are used up.  softmax: the weights are the
// softmax over the chosen scores, else the scores themselves.
__device__ __forceinline__ void choose_top(float* score, int E, int top, bool softmax, int lane, int* experts, float* weights) {
  float first = 0.f, sum = 0.f;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
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
      score[at] = -INFINITY;
    }
    if (j == 0) first = best;
    sum += expf(best - first);
    __syncwarp();
  }
  if (softmax)
    for (int j = lane; j < top; j += 32) weights[j] = expf(weights[j] - first) / sum;
}

// What the choice goes by beside the scores.
struct RouterGroups {
  const float* correction;  // [E]; null: none
  int groups, keep;
  __device__ __host__ bool plain() const { return correction == nullptr && groups == 1; }
};

// The same from choice[e] = score + correction within groups; score[e] is the weight, worth [groups] is scratch.  An expert's place is the
// number of better ones, so every place is taken once (NaN counts as the smallest number).
__device__ __forceinline__ void choose_grouped(float* choice, const float* score, float* worth, const RouterGroups& z, int E, int top, int lane,
                                               int* experts, float* weights) {
  constexpr float kLeast = -3.402823466e38f;
  for (int e = lane; e < E; e += 32) choice[e] = fmaxf(score[e] + (z.correction != nullptr ? z.correction[e] : 0.f), kLeast);
  __syncwarp();
  if (z.groups > 1) {
    const int size = E / z.groups;
    for (int g = lane; g < z.groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;                 // the best and the second
      for (int e = g * size; e < (g + 1) * size; ++e) {
        const float v = choice[e];
        b = fmaxf(b, fminf(a, v));
        a = fmaxf(a, v);
      }
      worth[g] = size > 1 ? fmaxf(a + b, kLeast) : a;
    }
    __syncwarp();
    for (int g = lane; g < z.groups; g += 32) {
      int better = 0;
      for (int i = 0; i < z.groups; ++i) better += worth[i] > worth[g] || (worth[i] == worth[g] && i < g);
      if (better >= z.keep)
        for (int e = g * size; e < (g + 1) * size; ++e) choice[e] = -INFINITY;
    }
    __syncwarp();
  }
  for (int e = lane; e < E; e += 32) {
    const float v = choice[e];
    if (v == -INFINITY) continue;
    int better = 0;
    for (int i = 0; i < E; ++i) better += choice[i] > v || (choice[i] == v && i < e);
    if (better < top) {
      experts[better] = e;
      weights[better] = score[e];
    }
  }
}

// bf16, W a multiple of 32, E <= 256: CTA = 16 MT tokens, the eight warps split W.  The order of the columns in a dot product is
// free, so a lane loads eight consecutive columns of its row (16 bytes) and uses them as the four column pairs of two mma
// k-steps, for tokens and experts alike: no shared memory on the way in.  The warps' partial logits are added in a fixed order.
template <int MT>
__global__ void __launch_bounds__(256) router_mma_kernel(const bf16* __restrict__ h, const bf16* __restrict__ w, int T, int W, int E, int top, bool softmax,
                                                         const RouterGroups groups, int* __restrict__ experts, float* __restrict__ weights) {
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
      score[e] = softmax ? z : 1.f / (1.f + expf(-z));
    }
    __syncwarp();
    int* chosen = experts + static_cast<size_t>(t0 + t) * top;
    float* weigh = weights + static_cast<size_t>(t0 + t) * top;
    if (groups.plain())
      choose_top(score, E, top, softmax, lane, chosen, weigh);
    else                                            // the token's other partial logits have been added up: their places are free
      choose_grouped(score + static_cast<size_t>(kTok) * Ep, score, score + static_cast<size_t>(2 * kTok) * Ep, groups, E, top, lane, chosen, weigh);
  }
}

// CTA = one token; one warp per expert at a time.
template <typename T, int N>
__global__ void __launch_bounds__(256) router_kernel(const T* __restrict__ h, const T* __restrict__ w, int W, int E, int top, bool softmax,
                                                     const RouterGroups groups, int* __restrict__ experts, float* __restrict__ weights) {
  extern __shared__ float score[];                  // [E]; with groups or corrections [3][E]
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* row = h + t * W;
  for (int e = warp; e < E; e += blockDim.x >> 5) {
    const T* we = w + static_cast<size_t>(e) * W;
    float z = 0.f;
#pragma unroll 4
    for (int i = lane * N; i < W; i += 32 * N) {
      float a[N], b[N];
      load_n<N>(row + i, a);
      load_n<N>(we + i, b);
#pragma unroll
      for (int q = 0; q < N; ++q) z = fmaf(a[q], b[q], z);
    }
    z = warp_sum_f(z);
    if (lane == 0) score[e] = softmax ? z : 1.f / (1.f + expf(-z));
  }
  __syncthreads();
  if (warp != 0) return;
  if (groups.plain()) choose_top(score, E, top, softmax, lane, experts + t * top, weights + t * top);
  else choose_grouped(score + E, score, score + 2 * E, groups, E, top, lane, experts + t * top, weights + t * top);
}

extern "C" int forge_router(int fp32, const void* h, const void* w, int T_, int W, int E, int top, int softmax, const float* correction,
                            int num_groups, int keep, int* experts, float* weights, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (E > 4096 || top < 1 || top > E) return -1;
  const RouterGroups groups = {correction, num_groups, keep};
  if (num_groups < 1 || E % num_groups || keep < 1 || keep > num_groups || top > keep * (E / num_groups) || (softmax && !groups.plain())) return -1;
  const bool v4 = (W & 3) == 0;
  const size_t smem = static_cast<size_t>(E) * 4 * (groups.plain() ? 1 : 3);      // at most 48 KB
  if (fp32) {
    auto k = v4 ? router_kernel<float, 4> : router_kernel<float, 1>;
    return launch_kernel(k, dim3(T_), dim3(256), smem, stream, 0, static_cast<const float*>(h), static_cast<const float*>(w), W, E, top, softmax != 0, groups, experts, weights) == cudaSuccess ? 0 : -2;
  }
  const bool aligned = ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
  // a few tokens would occupy a few CTAs of the kernel below: one CTA per token spreads them
  if (T_ <= 128 && (W & 7) == 0 && aligned)
    return launch_kernel(router_kernel<bf16, 8>, dim3(T_), dim3(256), smem, stream, 0, static_cast<const bf16*>(h), static_cast<const bf16*>(w), W, E, top, softmax != 0, groups, experts, weights) == cudaSuccess ? 0 : -2;
  if (W % 32 == 0 && E <= 256 && (reinterpret_cast<uintptr_t>(h) & 15) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0) {
    const int Ep = (E + 7) & ~7;
    const bool two = T_ > 2048 && E <= 128;        // more tokens per CTA halve the reads of the router matrix
    const dim3 grid((T_ + (two ? 31 : 15)) / (two ? 32 : 16));
    const size_t part = static_cast<size_t>(8) * (two ? 32 : 16) * Ep * 4;
    if (two) {
      FORGE_ENSURE_DYN_SMEM(router_mma_kernel<2>, 8 * 32 * 128 * 4);
      return launch_kernel(router_mma_kernel<2>, grid, dim3(256), part, stream, 0, static_cast<const bf16*>(h), static_cast<const bf16*>(w), T_, W, E, top, softmax != 0, groups, experts, weights) == cudaSuccess ? 0 : -2;
    }
    FORGE_ENSURE_DYN_SMEM(router_mma_kernel<1>, 8 * 16 * 256 * 4);
    return launch_kernel(router_mma_kernel<1>, grid, dim3(256), part, stream, 0, static_cast<const bf16*>(h), static_cast<const bf16*>(w), T_, W, E, top, softmax != 0, groups, experts, weights) == cudaSuccess ? 0 : -2;
  }
  auto k = v4 ? router_kernel<bf16, 4> : router_kernel<bf16, 1>;
  return launch_kernel(k, dim3(T_), dim3(256), smem, stream, 0, static_cast<const bf16*>(h), static_cast<const bf16*>(w), W, E, top, softmax != 0, groups, experts, weights) == cudaSuccess ? 0 : -2;
}

constexpr int kPlanThreads = 1024;

// One CTA.  smem: counts [E], next row [E].
__global__ void __launch_bounds__(kPlanThreads) moe_plan_kernel(const int* __restrict__ experts, int n, int E, int tile, int max_tiles,
                                                                int* __restrict__ pos, int* __restrict__ tile_expert,
                                                                int* __restrict__ num_tiles) {
  extern __shared__ int sm_plan[];
  int* count = sm_plan;
  int* next = sm_plan + E;
  pdl_launch_dependents();
  pdl_wait();
  for (int e = threadIdx.x; e < E; e += kPlanThreads) count[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += kPlanThreads) atomicAdd(&count[experts[i]], 1);
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
    for (int k = 0; k < (count[e] + tile - 1) / tile; ++k) tile_expert[next[e] / tile + k] = e;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += kPlanThreads) pos[i] = atomicAdd(&next[experts[i]], 1);
}

// max_tiles >= n / tile + E rounded up: the caller's buffer has max_tiles * tile rows.
extern "C" int forge_moe_plan(const int* experts, int n, int E, int tile, int max_tiles, int* pos, int* tile_expert, int* num_tiles,
                              cudaStream_t stream) {
  if (n <= 0) return 0;
  if (E > 4096 || tile < 1) return -1;
  return launch_kernel(moe_plan_kernel, dim3(1), dim3(kPlanThreads), static_cast<size_t>(E) * 8, stream, 0, experts, n, E, tile, max_tiles,
                       pos, tile_expert, num_tiles) == cudaSuccess ? 0 : -2;
}

template <typename T, int N>
__global__ void __launch_bounds__(256) moe_scatter_kernel(const T* __restrict__ h, const int* __restrict__ pos,
                                                          const float* __restrict__ weights, int top, int W, T* __restrict__ xs) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  for (int c = threadIdx.x * N; c < W; c += blockDim.x * N) {
    float v[N];
    load_n<N>(h + t * W + c, v);
    for (int j = 0; j < top; ++j) {
      const float s = weights != nullptr ? weights[t * top + j] : 1.f;
      float x[N];
#pragma unroll
      for (int e = 0; e < N; ++e) x[e] = s * v[e];
      store_n<N>(xs + static_cast<size_t>(pos[t * top + j]) * W + c, x);
    }
  }
}

extern "C" int forge_moe_scatter(int fp32, const void* h, const int* pos, const float* weights, int n, int top, int W, void* xs,
                                 cudaStream_t stream) {
  if (n <= 0) return 0;
  const bool v4 = (W & 3) == 0;
  if (fp32) {
    auto k = v4 ? moe_scatter_kernel<float, 4> : moe_scatter_kernel<float, 1>;
    return launch_kernel(k, dim3(n / top), dim3(256), 0, stream, 0, static_cast<const float*>(h), pos, weights, top, W, static_cast<float*>(xs)) == cudaSuccess ? 0 : -2;
  }
  auto k = v4 ? moe_scatter_kernel<bf16, 4> : moe_scatter_kernel<bf16, 1>;
  return launch_kernel(k, dim3(n / top), dim3(256), 0, stream, 0, static_cast<const bf16*>(h), pos, weights, top, W, static_cast<bf16*>(xs)) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
