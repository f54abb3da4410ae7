// Element types of kernels that exist in bf16 and in fp32 (a model that is served in 32-bit uses the fp32 instances):
// loads to fp32, stores from fp32, four elements at a time where alignment allows, and block sums.
#pragma once

#include "ptx.cuh"

namespace forge {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float load_f(const float* p) { return *p; }
__device__ __forceinline__ float load_f(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void store_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_f(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

// N consecutive elements (N = 1, 4 or 8; 4 fp32 or 8 bf16 need 16-byte alignment, 4 bf16 8-byte).
template <int N>
__device__ __forceinline__ void load_n(const float* p, float* v) {
  if constexpr (N == 8) {
    load_n<4>(p, v);
    load_n<4>(p + 4, v + 4);
  } else if constexpr (N == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else {
    v[0] = *p;
  }
}
template <int N>
__device__ __forceinline__ void load_n(const bf16* p, float* v) {
  if constexpr (N == 8) {
    const uint4 a = *reinterpret_cast<const uint4*>(p);
    v[0] = bf16_lo(a.x); v[1] = bf16_hi(a.x); v[2] = bf16_lo(a.y); v[3] = bf16_hi(a.y);
    v[4] = bf16_lo(a.z); v[5] = bf16_hi(a.z); v[6] = bf16_lo(a.w); v[7] = bf16_hi(a.w);
  } else if constexpr (N == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    v[0] = bf16_lo(a.x); v[1] = bf16_hi(a.x); v[2] = bf16_lo(a.y); v[3] = bf16_hi(a.y);
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int N>
__device__ __forceinline__ void store_n(float* p, const float* v) {
  if constexpr (N == 8) {
    store_n<4>(p, v);
    store_n<4>(p + 4, v + 4);
  } else if constexpr (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int N>
__device__ __forceinline__ void store_n(bf16* p, const float* v) {
  if constexpr (N == 8)
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  else if constexpr (N == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  else *p = __float2bfloat16_rn(v[0]);
}

__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Sum over the block; every thread gets it.  red: 32 floats of shared memory, free again on return.
__device__ __forceinline__ float block_sum_f(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum_f(v);
  if (lane == 0) red[warp] = v;
  __syncthreads();
  const float t = warp_sum_f(lane < nw ? red[lane] : 0.f);
  __syncthreads();
  return t;
}

// x * sigmoid(x) with the accurate exponential and division (fp32 instances) or the fast ones (bf16 instances).
template <typename T>
__device__ __forceinline__ float silu_t(float x) {
  if constexpr (sizeof(T) == 4) return x / (1.f + expf(-x));
  else return silu(x);
}

template <typename T>
__device__ __forceinline__ float sigmoid_t(float x) {
  if constexpr (sizeof(T) == 4) return 1.f / (1.f + expf(-x));
  else return __fdividef(1.f, 1.f + __expf(-x));
}

// log(1 + e^x) without overflow.
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// x = hi + lo with both halves in bf16 (|x - hi - lo| <= 2^-17 |x|): an fp32 factor as two tensor-core operands.
__device__ __forceinline__ void split_bf16(float x, float& hi, float& lo) {
  hi = __bfloat162float(__float2bfloat16_rn(x));
  lo = x - hi;
}

}  // namespace forge
