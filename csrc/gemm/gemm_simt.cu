// out = x w^T on the CUDA cores with fp32 accumulation, for what the tcgen05 GEMMs do not cover: fp32 operands (true 32-bit
// products) and bf16 shapes TMA cannot address (rows that are not a multiple of 16 bytes).
//
//   batch      blockIdx.z selects one of several independent products (per-head matrices)
//   experts    tile_expert[i] names the matrix that the 64-row tile i of x is multiplied with (< 0: tile not in use)
//
// Tiles of 64 x 64, 16 columns of K at a time, 4 x 4 outputs per thread; every bound is checked.
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kSB = 64, kSK = 16;

template <typename T>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const T* __restrict__ x, long long ldx, long long x_batch,
                                                        const T* __restrict__ w, long long ldw, long long w_batch,
                                                        T* __restrict__ out, long long ldo, long long o_batch, int M, int N, int K,
                                                        const int* __restrict__ tile_expert) {
  __shared__ float sx[kSK][kSB + 4];
  __shared__ float sw[kSK][kSB + 4];
  pdl_launch_dependents();
  pdl_wait();
  x += blockIdx.z * x_batch;
  out += blockIdx.z * o_batch;
  const int m0 = blockIdx.y * kSB, n0 = blockIdx.x * kSB;
  long long which = blockIdx.z;
  if (tile_expert != nullptr) {
    which = tile_expert[blockIdx.y];
    if (which < 0) return;
  }
  w += which * w_batch;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kSK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + i * 256, r = idx >> 4, c = idx & 15;
      const bool kin = k0 + c < K;
      sx[c][r] = kin && m0 + r < M ? load_f(x + (m0 + r) * ldx + k0 + c) : 0.f;
      sw[c][r] = kin && n0 + r < N ? load_f(w + (n0 + r) * ldw + k0 + c) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sx[k][ty * 4]), b = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (m0 + ty * 4 + i < M && n0 + tx * 4 + j < N) store_f(out + (m0 + ty * 4 + i) * ldo + n0 + tx * 4 + j, acc[i][j]);
}

// x [M, K] (row stride ldx), w [N, K], out [M, N]; `batch` products with the given element offsets between them.
extern "C" int forge_gemm_simt(int fp32, const void* x, long long ldx, long long x_batch, const void* w, long long ldw, long long w_batch,
                               void* out, long long ldo, long long o_batch, int M, int N, int K, int batch, const int* tile_expert,
                               cudaStream_t stream) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  const dim3 grid((N + kSB - 1) / kSB, (M + kSB - 1) / kSB, batch);
  if (grid.y > 65535 || grid.z > 65535) return -1;
  if (fp32)
    return launch_kernel(gemm_simt_kernel<float>, grid, dim3(256), 0, stream, 0, static_cast<const float*>(x), ldx, x_batch,
                         static_cast<const float*>(w), ldw, w_batch, static_cast<float*>(out), ldo, o_batch, M, N, K, tile_expert) == cudaSuccess ? 0 : -2;
  return launch_kernel(gemm_simt_kernel<bf16>, grid, dim3(256), 0, stream, 0, static_cast<const bf16*>(x), ldx, x_batch,
                       static_cast<const bf16*>(w), ldw, w_batch, static_cast<bf16*>(out), ldo, o_batch, M, N, K, tile_expert) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
