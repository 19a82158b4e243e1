// A norm on a sublayer's OUTPUT, added to the residual in the same launch:
//
//   x <- x + gain * y / sqrt(mean(y^2) + eps)
//
// x float32 [T, d] (in place), y [T, d] in the run dtype, gain float32 [d] (a checkpoint that stores
// it around zero has the one already added); optionally a copy of the new x in the run dtype, which is
// what the next sublayer's product reads.  Statistics and the sum are float32.
//
// One block a row.  Rows of a multiple of four elements stay in registers: a thread requests all its
// pieces of y and x (16 and 8 bytes each) before the reduction, so one round trip to memory serves
// both; the gains, which do not depend on the step, are requested ahead of the wait for the kernel
// before.  Other rows go through shared memory, an element at a time.
//
// norm_add_norm: the same sum followed at once by the norm that the next sublayer reads (layers with a norm
// before and after each sublayer):
//
//   x <- x + gain_b * y / sqrt(mean(y^2) + eps_b),   out = gain * x / sqrt(mean(x^2) + eps)
//
// with y = scale_1 y1 + scale_2 y2, the second optional (a mixer of two branches), formed in float32.  With a
// list of rows, output row i is made from batch row rows[i] and x is left alone (the final norm).
#include "common.cuh"
#include "pdl.cuh"

using namespace pbe;

namespace {

__device__ __forceinline__ void load4(const float* p, float (&a)[4]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  a[0] = v.x; a[1] = v.y; a[2] = v.z; a[3] = v.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&a)[4]) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  a[0] = lo.x; a[1] = lo.y; a[2] = hi.x; a[3] = hi.y;
}
__device__ __forceinline__ void store4(float* p, const float (&a)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(a[0], a[1], a[2], a[3]);
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&a)[4]) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a[0], a[1]), hi = __floats2bfloat162_rn(a[2], a[3]);
  uint2 raw;
  raw.x = *reinterpret_cast<const unsigned*>(&lo);
  raw.y = *reinterpret_cast<const unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = raw;
}

// VPT: groups of four elements a thread holds
template <typename T, int VPT>
__global__ void norm_add_kernel(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ gain,
                                T* __restrict__ lp, int d, float eps) {
  __shared__ float red[33];
  pdl_launch_dependents();
  float g[VPT][4];
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < d) load4(gain + i, g[j]);
  }
  pdl_wait();
  const size_t row = (size_t)blockIdx.x * d;
  float yv[VPT][4], xv[VPT][4];
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < d) {
      load4(y + row + i, yv[j]);
      load4(x + row + i, xv[j]);
    } else {
      yv[j][0] = yv[j][1] = yv[j][2] = yv[j][3] = 0.f;
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < VPT; ++j)
#pragma unroll
    for (int k = 0; k < 4; ++k) ss = fmaf(yv[j][k], yv[j][k], ss);
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps);
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < d) {
#pragma unroll
      for (int k = 0; k < 4; ++k) xv[j][k] += (yv[j][k] * inv) * g[j][k];
      store4(x + row + i, xv[j]);
      if (lp) store4(lp + row + i, xv[j]);
    }
  }
}

// any width: the row of y waits in shared memory
template <typename T>
__global__ void norm_add_any_kernel(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ gain,
                                    T* __restrict__ lp, int d, float eps) {
  __shared__ float red[33];
  extern __shared__ __align__(16) float held[];
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = (size_t)blockIdx.x * d;
  float ss = 0.f;
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    const float v = to_float(y[row + i]);
    held[i] = v;
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps);
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    const float v = x[row + i] + (held[i] * inv) * gain[i];
    x[row + i] = v;
    if (lp) lp[row + i] = from_float<T>(v);
  }
}

template <typename T>
int launch(float* x, const void* y, const float* gain, void* lp, int rows, int d, float eps, cudaStream_t stream) {
  const int groups = d / 4;
  if ((d & 3) == 0 && groups <= 4 * 1024) {
    if (groups <= 256) {
      launch_k(norm_add_kernel<T, 1>, rows, (groups + 31) / 32 * 32, 0, stream, x, (const T*)y, gain, (T*)lp, d, eps);
    } else {
      const int threads = ((groups + 3) / 4 + 31) / 32 * 32;
      launch_k(norm_add_kernel<T, 4>, rows, threads, 0, stream, x, (const T*)y, gain, (T*)lp, d, eps);
    }
    return launch_status();
  }
  const size_t smem = (size_t)d * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(norm_add_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  launch_k(norm_add_any_kernel<T>, rows, d >= 2048 ? 512 : 128, smem, stream, x, (const T*)y, gain, (T*)lp, d, eps);
  return launch_status();
}

struct ChainParams {
  float* x;                  // [T, d]
  const void* y1;            // [T, d]
  const void* y2;            // [T, d] or null
  float s1, s2;
  const float* gain_b;       // [d]
  const float* gain;         // [d]
  void* out;                 // [rows, d]
  const int32_t* rows;       // or null
  int d;
  float eps_b, eps;
};

template <typename T, int VPT>
__global__ void norm_add_norm_kernel(ChainParams p) {
  __shared__ float red[33];
  pdl_launch_dependents();
  const int d = p.d;
  float gb[VPT][4], g[VPT][4];
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < d) {
      load4(p.gain_b + i, gb[j]);
      load4(p.gain + i, g[j]);
    }
  }
  pdl_wait();
  const size_t row = (size_t)(p.rows ? p.rows[blockIdx.x] : (int)blockIdx.x) * d;
  float yv[VPT][4], xv[VPT][4];
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < d) {
      load4((const T*)p.y1 + row + i, yv[j]);
      load4(p.x + row + i, xv[j]);
#pragma unroll
      for (int k = 0; k < 4; ++k) yv[j][k] *= p.s1;
      if (p.y2) {
        float z[4];
        load4((const T*)p.y2 + row + i, z);
#pragma unroll
        for (int k = 0; k < 4; ++k) yv[j][k] = fmaf(p.s2, z[k], yv[j][k]);
      }
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k) yv[j][k] = xv[j][k] = 0.f;
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < VPT; ++j)
#pragma unroll
    for (int k = 0; k < 4; ++k) ss = fmaf(yv[j][k], yv[j][k], ss);
  const float inv_b = 1.0f / sqrtf(block_sum(ss, red) / (float)d + p.eps_b);
  ss = 0.f;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < d) {
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        xv[j][k] += (yv[j][k] * inv_b) * gb[j][k];
        ss = fmaf(xv[j][k], xv[j][k], ss);
      }
      if (!p.rows) store4(p.x + row + i, xv[j]);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + p.eps);
  T* out = (T*)p.out + (size_t)blockIdx.x * d;
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < d) {
#pragma unroll
      for (int k = 0; k < 4; ++k) xv[j][k] = (xv[j][k] * inv) * g[j][k];
      store4(out + i, xv[j]);
    }
  }
}

template <typename T>
__global__ void norm_add_norm_any_kernel(ChainParams p) {
  __shared__ float red[33];
  extern __shared__ __align__(16) float held[];
  pdl_launch_dependents();
  pdl_wait();
  const int d = p.d;
  const size_t row = (size_t)(p.rows ? p.rows[blockIdx.x] : (int)blockIdx.x) * d;
  float ss = 0.f;
  for (int i = threadIdx.x; i < d; i += blockDim.x) {
    float v = to_float(((const T*)p.y1)[row + i]) * p.s1;
    if (p.y2) v = fmaf(p.s2, to_float(((const T*)p.y2)[row + i]), v);
    held[i] = v;
    ss = fmaf(v, v, ss);
  }
  const float inv_b = 1.0f / sqrtf(block_sum(ss, red) / (float)d + p.eps_b);
  ss = 0.f;
  for (int i = threadIdx.x; i < d; i += blockDim.x) {      // a thread meets its own elements only
    const float v = p.x[row + i] + (held[i] * inv_b) * p.gain_b[i];
    held[i] = v;
    if (!p.rows) p.x[row + i] = v;
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + p.eps);
  T* out = (T*)p.out + (size_t)blockIdx.x * d;
  for (int i = threadIdx.x; i < d; i += blockDim.x) out[i] = from_float<T>((held[i] * inv) * p.gain[i]);
}

template <typename T>
int launch_chain(const ChainParams& p, int rows, cudaStream_t stream) {
  const int d = p.d, groups = d / 4;
  if ((d & 3) == 0 && groups <= 4 * 1024) {
    if (groups <= 256) {
      launch_k(norm_add_norm_kernel<T, 1>, rows, (groups + 31) / 32 * 32, 0, stream, p);
    } else if (groups <= 1024) {
      launch_k(norm_add_norm_kernel<T, 2>, rows, ((groups + 1) / 2 + 31) / 32 * 32, 0, stream, p);
    } else {
      launch_k(norm_add_norm_kernel<T, 4>, rows, ((groups + 3) / 4 + 31) / 32 * 32, 0, stream, p);
    }
    return launch_status();
  }
  const size_t smem = (size_t)d * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(norm_add_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  launch_k(norm_add_norm_any_kernel<T>, rows, d >= 2048 ? 512 : 128, smem, stream, p);
  return launch_status();
}
}  // namespace

PBE_EXPORT int pbe_norm_add(float* x, const void* y, int dtype, const float* gain, void* lp, int rows, int d, float eps,
                            cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (d < 1) return (int)cudaErrorInvalidValue;
  // sixteen-byte pieces of float32 rows, eight-byte pieces of bfloat16 rows
  if ((((uintptr_t)x | (uintptr_t)gain) & 15) || (((uintptr_t)y | (uintptr_t)lp) & (dtype == PBE_F32 ? 15 : 7)))
    return (int)cudaErrorMisalignedAddress;
  return dtype == PBE_F32 ? launch<float>(x, y, gain, lp, rows, d, eps, stream)
                          : launch<__nv_bfloat16>(x, y, gain, lp, rows, d, eps, stream);
}

PBE_EXPORT int pbe_norm_add_norm(float* x, const void* y1, const void* y2, float s1, float s2, int dtype,
                                 const float* gain_b, float eps_b, const float* gain, float eps, void* out,
                                 const int32_t* row_index, int rows, int d, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (d < 1) return (int)cudaErrorInvalidValue;
  if ((((uintptr_t)x | (uintptr_t)gain | (uintptr_t)gain_b) & 15) ||
      (((uintptr_t)y1 | (uintptr_t)y2 | (uintptr_t)out) & (dtype == PBE_F32 ? 15 : 7)))
    return (int)cudaErrorMisalignedAddress;
  ChainParams p{x, y1, y2, s1, s2, gain_b, gain, out, row_index, d, eps_b, eps};
  return dtype == PBE_F32 ? launch_chain<float>(p, rows, stream) : launch_chain<__nv_bfloat16>(p, rows, stream);
}
