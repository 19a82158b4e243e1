// Shared device helpers for the sm_100a kernels of this engine.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define PBE_EXPORT extern "C" __attribute__((visibility("default")))

// dtype codes shared with the Python side
#define PBE_F32 0
#define PBE_BF16 1

namespace pbe {

__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result.  The order of the
// additions is fixed by the thread layout, so a row's statistic does not depend on what
// else is in the batch.
__device__ __forceinline__ float block_sum(float v, float* smem /* >= 33 floats */) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) smem[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nwarps ? smem[lane] : 0.f;
    t = warp_sum(t);
    if (lane == 0) smem[32] = t;
  }
  __syncthreads();
  return smem[32];
}

// gelu in its tanh form, 0.5 z (1 + tanh(t)) with t = sqrt(2/pi) (z + 0.044715 z^3); since
// (1 + tanh t) / 2 = 1 / (1 + e^(-2t)) it is z times a sigmoid.  The fast form (for results that are
// rounded to bfloat16) takes the fast exponential and division.
__device__ __forceinline__ float gelu_tanh(float z) {
  const float t2 = 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);
  return z / (1.0f + expf(-t2));
}
__device__ __forceinline__ float gelu_tanh_fast(float z) {
  const float t2 = 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);
  return z * __fdividef(1.0f, 1.0f + __expf(-t2));
}

inline int launch_status() { return (int)cudaGetLastError(); }

}  // namespace pbe
