// Elementwise GEMM epilogues of the mixer stack, shared by the two tcgen05 GEMM kernels (their accumulator layouts differ:
// the general kernel holds 32 columns of one row per thread, the kernel for few tokens one column of 32 rows, or four
// columns of a row when it folds K splits).
#pragma once
#include "mixers.h"
#include "tcgen05_common.cuh"

namespace vb {

// tanh with fp32 accuracy in files compiled with fast math, without branches: the exponential form, and the first terms of
// the Maclaurin series near zero, where the former cancels.
__device__ __forceinline__ float tanh_full(float x) {
  const float ax = fabsf(x), s = x * x;
  const float small = x * (1.f + s * (-1.f / 3.f + s * (2.f / 15.f)));
  const float large = copysignf(1.f - __fdividef(2.f, 1.f + __expf(2.f * fminf(ax, 20.f))), x);
  return ax < 0.1f ? small : large;
}
__device__ __forceinline__ float gelu_erf_full(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }

__device__ __forceinline__ float silu_full(float z) { return z / (1.f + __expf(-z)); }
__device__ __forceinline__ float relu2(float z) { return fmaxf(z, 0.f) * fmaxf(z, 0.f); }

struct EpiColumn { float w, b, pw, pb; };  // weight and bias of an output column: of the norm of the stream, of the norm of the product
__device__ __forceinline__ EpiColumn epi_column(const VbEpiArgs& e, int col) {
  EpiColumn c{0.f, 0.f, 0.f, 0.f};
  if (e.mode == VB_EPI_RESID && e.D != nullptr) {
    c.w = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(e.nw)[col]);
    c.b = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(e.nb)[col]);
  }
  if (e.mode == VB_EPI_RESID && e.pw != nullptr) {
    c.pw = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(e.pw)[col]);
    c.pb = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(e.pb)[col]);
  }
  if (e.mode == VB_EPI_RESID && e.pw == nullptr && e.pb != nullptr) c.pb = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(e.pb)[col]);
  if (e.mode == VB_EPI_BIAS || e.mode == VB_EPI_BIAS_RELU2) c.b = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(e.nb)[col]);
  return c;
}
__device__ __forceinline__ float epi_palpha(const VbEpiArgs& e) {
  return (e.mode == VB_EPI_RESID && e.pw != nullptr) ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(e.palpha)) : 0.f;
}
__device__ __forceinline__ float epi_alpha(const VbEpiArgs& e) {
  return (e.mode == VB_EPI_RESID && e.D != nullptr) ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(e.alpha)) : 0.f;
}

// One element.
__device__ __forceinline__ void epi_store1(const VbEpiArgs& e, long long row, int col, float v, float alpha, float palpha, const EpiColumn& c) {
  __nv_bfloat16* D = reinterpret_cast<__nv_bfloat16*>(e.D);
  if (e.mode == VB_EPI_GELU) {
    D[row * e.ldd + col] = __float2bfloat16(gelu_erf_full(v));
  } else if (e.mode == VB_EPI_SOFTCAP) {
    D[row * e.ldd + col] = __float2bfloat16(e.cap * tanh_full(v / e.cap));
  } else if (e.mode == VB_EPI_STORE_F32) {
    reinterpret_cast<float*>(e.D)[row * e.ldd + col] = v;
  } else if (e.mode == VB_EPI_SPLIT) {
    if (col < e.n0) D[row * e.ldd + col] = __float2bfloat16(v);
    else e.D2[row * e.ldd2 + col - e.n0] = v;
  } else if (e.mode == VB_EPI_RESID) {
    const float x = e.X[row * e.ldx + col] + (e.pw != nullptr ? tanh_full(palpha * v) * c.pw + c.pb : v + c.pb);
    e.X[row * e.ldx + col] = x;
    if (D != nullptr) D[row * e.ldd + col] = __float2bfloat16(tanh_full(alpha * x) * c.w + c.b);
  } else if (e.mode == VB_EPI_BIAS) {
    D[row * e.ldd + col] = __float2bfloat16(v + c.b);
  } else if (e.mode == VB_EPI_SILU) {
    D[row * e.ldd + col] = __float2bfloat16(col < e.n0 ? silu_full(v) : v);
  } else if (e.mode == VB_EPI_BIAS_RELU2) {
    D[row * e.ldd + col] = __float2bfloat16(relu2(v + c.b));
  } else if (e.mode == VB_EPI_TANH) {
    D[row * e.ldd + col] = __float2bfloat16(col < e.n0 ? v : tanh_full(v));
  } else {
    D[row * e.ldd + col] = __float2bfloat16(v);
  }
}

// NV consecutive columns of one row (NV = 4 or 8, col a multiple of NV, split point a multiple of NV).
template <int NV>
__device__ __forceinline__ void epi_store_row(const VbEpiArgs& e, long long row, int col, const float (&v)[NV], float alpha, float palpha) {
  __nv_bfloat16* D = reinterpret_cast<__nv_bfloat16*>(e.D);
  auto put16 = [&](const float (&o)[NV]) {
    __nv_bfloat16* dst = D + row * e.ldd + col;
    if constexpr (NV == 8)
      *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16x2(o[0], o[1]), pack_bf16x2(o[2], o[3]), pack_bf16x2(o[4], o[5]), pack_bf16x2(o[6], o[7]));
    else
      *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(o[0], o[1]), pack_bf16x2(o[2], o[3]));
  };
  auto put32 = [&](float* dst, const float (&o)[NV]) {
#pragma unroll
    for (int i = 0; i < NV; i += 4) *reinterpret_cast<float4*>(dst + i) = make_float4(o[i], o[i + 1], o[i + 2], o[i + 3]);
  };
  if (e.mode == VB_EPI_GELU) {
    float o[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] = gelu_erf_full(v[i]);
    put16(o);
  } else if (e.mode == VB_EPI_SOFTCAP) {
    float o[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] = e.cap * tanh_full(v[i] / e.cap);
    put16(o);
  } else if (e.mode == VB_EPI_STORE_F32) {
    put32(reinterpret_cast<float*>(e.D) + row * e.ldd + col, v);
  } else if (e.mode == VB_EPI_SPLIT) {
    if (col < e.n0) put16(v);
    else put32(e.D2 + row * e.ldd2 + col - e.n0, v);
  } else if (e.mode == VB_EPI_RESID) {
    float* xp = e.X + row * e.ldx + col;
    float o[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] = v[i];
    if (e.pw != nullptr) {
      const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(e.pw) + col;
      const __nv_bfloat16* b = reinterpret_cast<const __nv_bfloat16*>(e.pb) + col;
#pragma unroll
      for (int i = 0; i < NV; ++i) o[i] = tanh_full(palpha * v[i]) * __bfloat162float(w[i]) + __bfloat162float(b[i]);
    } else if (e.pb != nullptr) {
      const __nv_bfloat16* b = reinterpret_cast<const __nv_bfloat16*>(e.pb) + col;
#pragma unroll
      for (int i = 0; i < NV; ++i) o[i] += __bfloat162float(b[i]);
    }
#pragma unroll
    for (int i = 0; i < NV; i += 4) {
      const float4 a = *reinterpret_cast<const float4*>(xp + i);
      o[i] += a.x; o[i + 1] += a.y; o[i + 2] += a.z; o[i + 3] += a.w;
    }
    put32(xp, o);
    if (D != nullptr) {
      const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(e.nw) + col;
      const __nv_bfloat16* b = reinterpret_cast<const __nv_bfloat16*>(e.nb) + col;
#pragma unroll
      for (int i = 0; i < NV; ++i) o[i] = tanh_full(alpha * o[i]) * __bfloat162float(w[i]) + __bfloat162float(b[i]);
      put16(o);
    }
  } else if (e.mode == VB_EPI_BIAS || e.mode == VB_EPI_BIAS_RELU2) {
    const __nv_bfloat16* b = reinterpret_cast<const __nv_bfloat16*>(e.nb) + col;
    float o[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] = v[i] + __bfloat162float(b[i]);
    if (e.mode == VB_EPI_BIAS_RELU2) {
#pragma unroll
      for (int i = 0; i < NV; ++i) o[i] = relu2(o[i]);
    }
    put16(o);
  } else if (e.mode == VB_EPI_TANH) {
    float o[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] = v[i];
    if (col + NV > e.n0) {
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (col + i >= e.n0) o[i] = tanh_full(v[i]);
    }
    put16(o);
  } else if (e.mode == VB_EPI_SILU) {
    float o[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] = col + i < e.n0 ? silu_full(v[i]) : v[i];
    put16(o);
  } else {
    put16(v);
  }
}

// Vector stores of `nv` columns need these alignments of the outputs.
inline bool epi_aligned(const VbEpiArgs& e, int nv) {
  auto bad = [](const void* p, int bytes) { return p != nullptr && (reinterpret_cast<uintptr_t>(p) % bytes) != 0; };
  const bool f32 = e.mode == VB_EPI_STORE_F32;
  if (e.D != nullptr && ((e.ldd % (f32 ? 4 : nv)) || bad(e.D, f32 ? 16 : 2 * nv))) return false;
  if (e.mode == VB_EPI_SPLIT && ((e.n0 % 8) || (e.ldd2 % 4) || bad(e.D2, 16))) return false;
  if (e.mode == VB_EPI_RESID && ((e.ldx % 4) || bad(e.X, 16) || bad(e.pw, 4) || bad(e.pb, 4) || (e.D != nullptr && (bad(e.nw, 4) || bad(e.nb, 4))))) return false;
  return true;
}

}  // namespace vb
