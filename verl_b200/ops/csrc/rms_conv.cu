// Row kernels of stacks with RMS norms in front of the sublayers: embedding, and norm of the residual stream with an optional causal
// convolution of its output over time, h + conv(h). A decode step's kernel also adds the partial products of the GEMM in front of it
// (and a bias) to the stream, takes the convolution's past from the slot's state and moves it on. Prompts: a CTA takes a run of
// consecutive tokens; statistics first (a warp per row), then every thread walks its columns through the run with the window of normed
// rows in registers. What a sequence keeps (fp32) is written by a second small launch. Compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>
#include <type_traits>

namespace vb {

typedef __nv_bfloat16 bf16;

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
embed_rows_kernel(const long long* __restrict__ ids, const T* __restrict__ w, float scale, float* __restrict__ x, int W, int V, long long total) {
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= total) return;
  const int per = W / VEC, c = static_cast<int>(i % per) * VEC;
  const long long t = i / per, id = ids[t];
  float v[VEC] = {};
  if (id >= 0 && id < V) Vec<T, VEC>::load(w + id * W + c, v);
#pragma unroll
  for (int k = 0; k < VEC; ++k) v[k] *= scale;
  Vec<float, VEC>::store(x + t * W + c, v);
}

// --------------------------------------------------------------------------------------------- one token per row
// One CTA per token; a thread keeps its ITEMS x VEC columns in registers between the two passes.
template <typename T, int VEC, int ITEMS>
__global__ void rms_rows_kernel(const VbRmsConv p) {
  __shared__ float red[33];
  const long long t = blockIdx.x;
  float x[ITEMS][VEC], v[VEC], ss = 0.f;
  float* xr = p.x + t * p.W;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
    if (c >= p.W) continue;
    Vec<float, VEC>::load(xr + c, x[it]);
    if (p.y != nullptr) {
      float y[VEC] = {};
      if (p.y_f32) {
        const float* src = reinterpret_cast<const float*>(p.y) + t * p.ldy + c;
        for (int s = 0; s < p.splits; ++s) {
          Vec<float, VEC>::load(src + s * p.split_stride, v);
#pragma unroll
          for (int i = 0; i < VEC; ++i) y[i] += v[i];
        }
      } else {
        Vec<T, VEC>::load(reinterpret_cast<const T*>(p.y) + t * p.ldy + c, y);
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[it][i] += y[i];
    }
    if (p.bias != nullptr) {
      Vec<T, VEC>::load(reinterpret_cast<const T*>(p.bias) + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[it][i] += v[i];
    }
    if (p.y != nullptr || p.bias != nullptr) Vec<float, VEC>::store(xr + c, x[it]);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += x[it][i] * x[it][i];
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / p.W + p.eps);
  const T *nw = reinterpret_cast<const T*>(p.nw), *conv = reinterpret_cast<const T*>(p.conv);
  T* hr = reinterpret_cast<T*>(p.h) + t * p.W;
  float* st = conv != nullptr && p.taps > 1 && p.state != nullptr && p.active[t] ? p.state + t * p.slot_stride : nullptr;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
    if (c >= p.W) continue;
    Vec<T, VEC>::load(nw + c, v);
    float o[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) o[i] = x[it][i] = x[it][i] * r * v[i];
    if (conv != nullptr) {
      for (int j = 0; j < p.taps; ++j) {
        const bool self = j == p.taps - 1;
        float past[VEC];
        if (!self) {
          if (st == nullptr) continue;
          Vec<float, VEC>::load(st + static_cast<long long>(j) * p.W + c, past);
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) o[i] += to_f(conv[static_cast<long long>(c + i) * p.taps + j]) * (self ? x[it][i] : past[i]);
        if (!self && j > 0) Vec<float, VEC>::store(st + static_cast<long long>(j - 1) * p.W + c, past);
      }
      if (st != nullptr) Vec<float, VEC>::store(st + static_cast<long long>(p.taps - 2) * p.W + c, x[it]);
    }
    Vec<T, VEC>::store(hr + c, o);
  }
}

template <typename T, int VEC>
static int rms_rows(const VbRmsConv* p, cudaStream_t s) {
  const int nvec = (p->W + VEC - 1) / VEC;
  int thr = nvec >= 256 ? 256 : (nvec + 31) / 32 * 32;
  if (nvec > 8 * thr) thr = 1024;
  const int items = (nvec + thr - 1) / thr;
  auto go = [&](auto kern) {
    kern<<<p->T, thr, 0, s>>>(*p);
    return static_cast<int>(cudaGetLastError());
  };
  if (items == 1) return go(rms_rows_kernel<T, VEC, 1>);
  if (items == 2) return go(rms_rows_kernel<T, VEC, 2>);
  if (items <= 4) return go(rms_rows_kernel<T, VEC, 4>);
  if (items <= 8) return go(rms_rows_kernel<T, VEC, 8>);
  if (items <= 32) return go(rms_rows_kernel<T, VEC, 32>);
  return -1;
}

// --------------------------------------------------------------------------------------------- portions with a convolution
__device__ __forceinline__ int rc_sequence(const VbRmsConv& a, long long t) {
  int lo = 0, hi = a.B - 1;
  while (lo < hi) {
    const int mid = (lo + hi) / 2;
    if (a.cu[mid + 1] <= t) lo = mid + 1; else hi = mid;
  }
  return lo;
}
// What the sequence kept (null: zeros).
__device__ __forceinline__ float* rc_past(const VbRmsConv& a, int b) {
  if (a.state == nullptr || a.slots == nullptr || a.slots[b] < 0 || (a.fresh != nullptr && a.fresh[b] != 0)) return nullptr;
  return a.state + static_cast<long long>(a.slots[b]) * a.slot_stride;
}
// 1 / root mean square of a row, every lane of the warp gets it
template <int VEC>
__device__ __forceinline__ float rc_scale(const float* x, int W, float eps) {
  const int lane = threadIdx.x & 31;
  float ss = 0.f, v[VEC];
  for (int c = lane * VEC; c < W; c += 32 * VEC) {
    Vec<float, VEC>::load(x + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += v[i] * v[i];
  }
  return 1.f / sqrtf(warp_sum(ss) / W + eps);
}

constexpr int RC_RUN = 16;   // tokens of a CTA
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(256)
rms_conv_kernel(const VbRmsConv a) {
  constexpr int PAST = TAPS - 1;
  __shared__ float inv[RC_RUN + PAST];               // of tokens t0 - PAST ..
  const int t0 = blockIdx.x * RC_RUN, t1 = min(a.T, t0 + RC_RUN), warp = threadIdx.x >> 5;
  for (int i = warp; i < t1 - t0 + PAST; i += 8) {
    const int t = t0 - PAST + i;
    const float f = t >= 0 ? rc_scale<VEC>(a.x + static_cast<long long>(t) * a.W, a.W, a.eps) : 0.f;
    if ((threadIdx.x & 31) == 0) inv[i] = f;
  }
  __syncthreads();
  const T *nw = reinterpret_cast<const T*>(a.nw), *conv = reinterpret_cast<const T*>(a.conv);
  T* h = reinterpret_cast<T*>(a.h);
  for (int c = threadIdx.x * VEC; c < a.W; c += 256 * VEC) {
    float g[VEC], w[TAPS][VEC], past[PAST > 0 ? PAST : 1][VEC];
    Vec<T, VEC>::load(nw + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[j][i] = to_f(conv[static_cast<long long>(c + i) * TAPS + j]);
    // the rows in front of token t: of its portion, then what the sequence kept, then zeros
    int end = 0;
    auto refill = [&](int t) {
      const int b = rc_sequence(a, t), back = t - a.cu[b];
      const float* st = back < PAST ? rc_past(a, b) : nullptr;
      end = a.cu[b + 1];
#pragma unroll
      for (int k = 0; k < PAST; ++k) {
        const int at = back - PAST + k;              // index inside the portion
#pragma unroll
        for (int i = 0; i < VEC; ++i) past[k][i] = 0.f;
        if (at >= 0) {
          Vec<float, VEC>::load(a.x + static_cast<long long>(t - PAST + k) * a.W + c, past[k]);
#pragma unroll
          for (int i = 0; i < VEC; ++i) past[k][i] *= inv[t - t0 + k] * g[i];
        } else if (st != nullptr) {
          Vec<float, VEC>::load(st + static_cast<long long>(at + PAST) * a.W + c, past[k]);
        }
      }
    };
    if (PAST > 0) refill(t0);
    constexpr int U = 4;                             // rows in flight
    for (int u0 = t0; u0 < t1; u0 += U) {
      float x[U][VEC];
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (u0 + u < t1) Vec<float, VEC>::load(a.x + static_cast<long long>(u0 + u) * a.W + c, x[u]);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int t = u0 + u;
        if (t >= t1) break;
        if (PAST > 0 && t >= end) refill(t);
        const float r = inv[t - t0 + PAST];
        float o[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          x[u][i] *= r * g[i];
          o[i] = x[u][i] + w[PAST][i] * x[u][i];
#pragma unroll
          for (int k = 0; k < PAST; ++k) o[i] += w[k][i] * past[k][i];
        }
        Vec<T, VEC>::store(h + static_cast<long long>(t) * a.W + c, o);
        if constexpr (PAST > 0) {
#pragma unroll
          for (int k = 0; k + 1 < PAST; ++k)
#pragma unroll
            for (int i = 0; i < VEC; ++i) past[k][i] = past[k + 1][i];
#pragma unroll
          for (int i = 0; i < VEC; ++i) past[PAST - 1][i] = x[u][i];
        }
      }
    }
  }
}

// Any number of taps: one CTA per token, the rows of the window are normed again.
template <typename T>
__global__ void __launch_bounds__(256)
rms_conv_any_kernel(const VbRmsConv a) {
  extern __shared__ float inv[];                     // [taps], of tokens t - past ..
  const int t = blockIdx.x, past = a.taps - 1, warp = threadIdx.x >> 5, b = rc_sequence(a, t), back = t - a.cu[b];
  const float* st = back < past ? rc_past(a, b) : nullptr;
  for (int j = warp; j < a.taps; j += 8) {
    const int s = t - past + j;
    const float f = s >= a.cu[b] ? rc_scale<1>(a.x + static_cast<long long>(s) * a.W, a.W, a.eps) : 0.f;
    if ((threadIdx.x & 31) == 0) inv[j] = f;
  }
  __syncthreads();
  const T *nw = reinterpret_cast<const T*>(a.nw), *conv = reinterpret_cast<const T*>(a.conv);
  for (int c = threadIdx.x; c < a.W; c += 256) {
    const float g = to_f(nw[c]);
    float o = a.x[static_cast<long long>(t) * a.W + c] * inv[past] * g;
    for (int j = 0; j < a.taps; ++j) {
      const int at = back - past + j;
      const float v = at >= 0 ? a.x[static_cast<long long>(t - past + j) * a.W + c] * inv[j] * g : (st != nullptr ? st[static_cast<long long>(at + past) * a.W + c] : 0.f);
      o += to_f(conv[static_cast<long long>(c) * a.taps + j]) * v;
    }
    reinterpret_cast<T*>(a.h)[static_cast<long long>(t) * a.W + c] = from_f<T>(o);
  }
}

// The last taps - 1 normed rows of every portion (a portion shorter than that moves older ones up). One CTA per sequence.
template <typename T>
__global__ void __launch_bounds__(256)
rms_conv_state_kernel(const VbRmsConv a) {
  extern __shared__ float inv[];                     // [taps - 1]
  const int b = blockIdx.x, past = a.taps - 1, warp = threadIdx.x >> 5;
  const int s0 = a.cu[b], n = a.cu[b + 1] - s0;
  if (a.slots[b] < 0 || n <= 0) return;
  const bool zero = a.fresh != nullptr && a.fresh[b] != 0;
  for (int j = warp; j < past; j += 8) {
    const int at = n - past + j;
    const float f = at >= 0 ? rc_scale<1>(a.x + static_cast<long long>(s0 + at) * a.W, a.W, a.eps) : 0.f;
    if ((threadIdx.x & 31) == 0) inv[j] = f;
  }
  __syncthreads();
  float* st = a.state + static_cast<long long>(a.slots[b]) * a.slot_stride;
  for (int c = threadIdx.x; c < a.W; c += 256) {
    const float g = to_f(reinterpret_cast<const T*>(a.nw)[c]);
    for (int j = 0; j < past; ++j) {
      const int at = n - past + j;                   // reads ahead of what it writes
      st[static_cast<long long>(j) * a.W + c] = at >= 0 ? a.x[static_cast<long long>(s0 + at) * a.W + c] * inv[j] * g
                                                        : (zero ? 0.f : st[static_cast<long long>(at + past) * a.W + c]);
    }
  }
}

template <typename T, int VEC>
static int rms_conv_run(const VbRmsConv* p, cudaStream_t s) {
  const unsigned grid = static_cast<unsigned>((p->T + RC_RUN - 1) / RC_RUN);
  if (p->taps == 1) rms_conv_kernel<T, VEC, 1><<<grid, 256, 0, s>>>(*p);
  else if (p->taps == 2) rms_conv_kernel<T, VEC, 2><<<grid, 256, 0, s>>>(*p);
  else if (p->taps == 3) rms_conv_kernel<T, VEC, 3><<<grid, 256, 0, s>>>(*p);
  else if (p->taps == 4) rms_conv_kernel<T, VEC, 4><<<grid, 256, 0, s>>>(*p);
  else if (p->taps <= 4096) rms_conv_any_kernel<T><<<p->T, 256, p->taps * 4, s>>>(*p);
  else return -1;
  return static_cast<int>(cudaGetLastError());
}

static bool rc_mis16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) != 0; }

}  // namespace vb

using namespace vb;

extern "C" int vb_embed_rows(int dtype, const long long* ids, const void* w, float scale, float* x, int T, int W, int V, cudaStream_t s) {
  if (T <= 0) return 0;
  const bool vec = W % 8 == 0 && !rc_mis16(w) && !rc_mis16(x);
  const long long total = static_cast<long long>(T) * (vec ? W / 8 : W);
  const unsigned grid = static_cast<unsigned>((total + 255) / 256);
  if (dtype == 0) {
    if (vec) embed_rows_kernel<float, 8><<<grid, 256, 0, s>>>(ids, (const float*)w, scale, x, W, V, total);
    else embed_rows_kernel<float, 1><<<grid, 256, 0, s>>>(ids, (const float*)w, scale, x, W, V, total);
  } else {
    if (vec) embed_rows_kernel<bf16, 8><<<grid, 256, 0, s>>>(ids, (const bf16*)w, scale, x, W, V, total);
    else embed_rows_kernel<bf16, 1><<<grid, 256, 0, s>>>(ids, (const bf16*)w, scale, x, W, V, total);
  }
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_rms_conv(int dtype, const VbRmsConv* p, cudaStream_t s) {
  if (p->T <= 0) return 0;
  const bool vec = p->W % 8 == 0 && p->ldy % 8 == 0 && p->split_stride % 8 == 0 && p->slot_stride % 4 == 0 && !rc_mis16(p->x) && !rc_mis16(p->y) && !rc_mis16(p->bias) &&
                   !rc_mis16(p->nw) && !rc_mis16(p->state) && !rc_mis16(p->h);
  if (p->conv == nullptr || p->cu == nullptr) {
    if (dtype == 0) return vec ? rms_rows<float, 8>(p, s) : rms_rows<float, 1>(p, s);
    return vec ? rms_rows<bf16, 8>(p, s) : rms_rows<bf16, 1>(p, s);
  }
  int rc;
  if (dtype == 0) rc = vec ? rms_conv_run<float, 8>(p, s) : rms_conv_run<float, 1>(p, s);
  else rc = vec ? rms_conv_run<bf16, 8>(p, s) : rms_conv_run<bf16, 1>(p, s);
  if (rc == 0 && p->state != nullptr && p->slots != nullptr && p->taps > 1) {
    if (dtype == 0) rms_conv_state_kernel<float><<<p->B, 256, p->taps * 4, s>>>(*p);
    else rms_conv_state_kernel<bf16><<<p->B, 256, p->taps * 4, s>>>(*p);
    rc = static_cast<int>(cudaGetLastError());
  }
  return rc;
}
