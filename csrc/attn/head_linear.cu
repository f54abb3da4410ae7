// Per-head products  out[t, h, :] = w[h] x[t, h, :]  (w [heads, N, K], K contiguous): the key matrix folded into the queries and
// the value matrix applied to the attended latents of a latent-attention decode step.  A CTA multiplies 64 tokens of one head by
// 32 rows of its matrix on mma.sync; K comes in 64 columns at a time through a three-stage cp.async ring.
#include "../include/launch.cuh"
#include "../include/mma_sync.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kHM = 64, kHN = 32, kHK = 64, kHPitch = kHK + 8, kHStages = 3;

__global__ void __launch_bounds__(128) head_linear_kernel(const bf16* __restrict__ x, long long x_tok, long long x_head,
                                                          const bf16* __restrict__ w, bf16* __restrict__ out, long long o_tok,
                                                          long long o_head, int M, int N, int K) {
  __shared__ __align__(16) bf16 sx[kHStages][kHM][kHPitch];
  __shared__ __align__(16) bf16 sw[kHStages][kHN][kHPitch];
  const int n0 = blockIdx.x * kHN, m0 = blockIdx.y * kHM, h = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  x += h * x_head;
  w += static_cast<size_t>(h) * N * K;
  out += h * o_head;
  const int num_kb = (K + kHK - 1) / kHK;
  auto load_w = [&](int kb) {                              // weights do not depend on the kernel before
    const int s = kb % kHStages, k0 = kb * kHK;
    for (int i = threadIdx.x; i < kHN * (kHK / 8); i += 128) {
      const int r = i >> 3, c = (i & 7) * 8;
      const bool in = n0 + r < N && k0 + c < K;
      cp_async16(smem_u32(&sw[s][r][c]), in ? w + static_cast<size_t>(n0 + r) * K + k0 + c : w, in ? 16 : 0);
    }
  };
  auto load_x = [&](int kb) {
    const int s = kb % kHStages, k0 = kb * kHK;
    for (int i = threadIdx.x; i < kHM * (kHK / 8); i += 128) {
      const int r = i >> 3, c = (i & 7) * 8;
      const bool in = m0 + r < M && k0 + c < K;
      cp_async16(smem_u32(&sx[s][r][c]), in ? x + (m0 + r) * x_tok + k0 + c : x, in ? 16 : 0);
    }
  };
  pdl_launch_dependents();
  for (int kb = 0; kb < kHStages - 1 && kb < num_kb; ++kb) load_w(kb);
  pdl_wait();
  for (int kb = 0; kb < kHStages - 1; ++kb) {
    if (kb < num_kb) load_x(kb);
    cp_async_commit();                                     // the weights issued above belong to the first group
  }
  float acc[kHN / 8][4] = {};
  for (int kb = 0; kb < num_kb; ++kb) {
    cp_async_wait<kHStages - 2>();
    __syncthreads();
    if (kb + kHStages - 1 < num_kb) {
      load_w(kb + kHStages - 1);
      load_x(kb + kHStages - 1);
    }
    cp_async_commit();
    const int s = kb % kHStages;
#pragma unroll
    for (int ks = 0; ks < kHK / 16; ++ks) {
      uint32_t a[4];
      ldsm_x4(smem_u32(&sx[s][warp * 16 + (lane & 15)][ks * 16 + (lane >> 4) * 8]), a);
#pragma unroll
      for (int nb = 0; nb < kHN / 8; nb += 2) {
        uint32_t b[4];
        ldsm_x4(smem_u32(&sw[s][nb * 8 + (lane & 7) + (lane >> 4) * 8][ks * 16 + ((lane >> 3) & 1) * 8]), b);
        mma16816(acc[nb], a, b[0], b[1]);
        mma16816(acc[nb + 1], a, b[2], b[3]);
      }
    }
  }
  const int r0 = m0 + warp * 16 + (lane >> 2);
#pragma unroll
  for (int nb = 0; nb < kHN / 8; ++nb) {
    const int c = n0 + nb * 8 + 2 * (lane & 3);
    if (c >= N) continue;                                  // N is even
    if (r0 < M) *reinterpret_cast<uint32_t*>(out + r0 * o_tok + c) = pack_bf16x2(acc[nb][0], acc[nb][1]);
    if (r0 + 8 < M) *reinterpret_cast<uint32_t*>(out + (r0 + 8) * o_tok + c) = pack_bf16x2(acc[nb][2], acc[nb][3]);
  }
}

// Strides in elements.  K, x strides and w rows: multiples of 8 (16-byte rows); N and out strides: even.
extern "C" int forge_head_linear(const void* x, long long x_tok, long long x_head, const void* w, void* out, long long o_tok,
                                 long long o_head, int M, int heads, int N, int K, cudaStream_t stream) {
  if (M <= 0) return 0;
  if ((K & 7) || (x_tok & 7) || (x_head & 7) || (N & 1) || (o_tok & 1) || (o_head & 1) || (reinterpret_cast<uintptr_t>(x) & 15) ||
      (reinterpret_cast<uintptr_t>(w) & 15) || (reinterpret_cast<uintptr_t>(out) & 3) || heads > 65535 || (M + kHM - 1) / kHM > 65535)
    return -1;
  return launch_kernel(head_linear_kernel, dim3((N + kHN - 1) / kHN, (M + kHM - 1) / kHM, heads), dim3(128), 0, stream, 0,
                       static_cast<const bf16*>(x), x_tok, x_head, static_cast<const bf16*>(w), static_cast<bf16*>(out), o_tok, o_head,
                       M, N, K) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
