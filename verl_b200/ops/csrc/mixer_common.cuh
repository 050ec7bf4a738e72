// Small device helpers shared by the mixer-stack kernels.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace vb {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
// log(sigmoid(z)) without overflow on either side
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

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
// Sum over the block; `red` holds at least 33 floats. Every thread gets the result.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[w] = v;
  __syncthreads();
  if (w == 0) {
    float t = (threadIdx.x & 31) < nw ? red[threadIdx.x & 31] : 0.f;
    t = warp_sum(t);
    if (threadIdx.x == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}

// VEC consecutive elements <-> floats
template <typename T, int VEC>
struct Vec;
template <int VEC>
struct Vec<float, VEC> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[VEC]) {
    if constexpr (VEC % 4 == 0) {
#pragma unroll
      for (int i = 0; i < VEC; i += 4) {
        const float4 a = *reinterpret_cast<const float4*>(p + i);
        v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
      }
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = p[i];
    }
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[VEC]) {
    if constexpr (VEC % 4 == 0) {
#pragma unroll
      for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) p[i] = v[i];
    }
  }
};
template <int VEC>
struct Vec<__nv_bfloat16, VEC> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[VEC]) {
    if constexpr (VEC == 8) {
      const uint4 a = *reinterpret_cast<const uint4*>(p);
      const uint32_t u[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[2 * i] = __uint_as_float(u[i] << 16);
        v[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
      }
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = __bfloat162float(p[i]);
    }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[VEC]) {
    if constexpr (VEC == 8) {
      uint32_t u[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        u[i] = *reinterpret_cast<uint32_t*>(&b);
      }
      *reinterpret_cast<uint4*>(p) = make_uint4(u[0], u[1], u[2], u[3]);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) p[i] = __float2bfloat16(v[i]);
    }
  }
};

}  // namespace vb
