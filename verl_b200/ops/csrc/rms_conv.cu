// Row kernels of stacks with RMS norms in front of the sublayers: embedding, and norm of the residual stream with an optional causal
// convolution of its output over time, h + conv(h). A decode step's kernel also adds the partial products of the GEMM in front of it
// (and a bias) to the stream, takes the convolution's past from the slot's state and moves it on. Prompts: a CTA walks a run of
// consecutive tokens, four at a time (the next four on their way), and keeps the window of normed rows in registers; rows too wide for
// that are read twice (statistics first, a warp per row). What a sequence keeps (fp32) is written by a second small launch. Compiled without fast math.
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

// Rows too wide for the kernel below, and columns one at a time.
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

// two floats in a register pair: one instruction for both
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("{\n.reg .b64 a, b, c, d;\nmov.b64 a, {%2, %3};\nmov.b64 b, {%4, %5};\nmov.b64 c, {%6, %7};\nfma.rn.f32x2 d, a, b, c;\nmov.b64 {%0, %1}, d;\n}"
      : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 d;
  asm("{\n.reg .b64 a, b, d;\nmov.b64 a, {%2, %3};\nmov.b64 b, {%4, %5};\nmul.rn.f32x2 d, a, b;\nmov.b64 {%0, %1}, d;\n}" : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}

// The same with every row read once: a thread owns eight columns (W <= 8 blockDim), four tokens share a reduction, the rows of the next
// eight are on their way to shared memory (every thread fetches and reads its own columns).
constexpr int RW_RUN = 16, RW_N = 4, RW_STAGES = 3, RW_VEC = 8;
template <typename T, int TAPS>
__global__ void __launch_bounds__(512)
rms_conv_once_kernel(const VbRmsConv a) {
  constexpr int PAST = TAPS - 1, H = RW_VEC / 2;
  extern __shared__ __align__(16) float ring[];      // [stage][token][thread][8]
  __shared__ float part[2][16][RW_N];
  const int t0 = blockIdx.x * RW_RUN, t1 = min(a.T, t0 + RW_RUN), warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, c = threadIdx.x * RW_VEC;
  const bool on = c < a.W;
  const int first = max(0, t0 - PAST);               // rows t0 - PAST .. are normed too
  float* mine = ring + threadIdx.x * RW_VEC;
  const int row = blockDim.x * RW_VEC;
  auto fetch = [&](int n) {                          // batch n
#pragma unroll
    for (int u = 0; u < RW_N; ++u) {
      const int t = first + n * RW_N + u;
      if (t < t1) {
        const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(mine + (n % RW_STAGES * RW_N + u) * row));
        const float* src = a.x + static_cast<long long>(t) * a.W + (on ? c : 0);
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(on ? 16 : 0) : "memory");
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + 16), "l"(src + 4), "r"(on ? 16 : 0) : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int n = 0; n < RW_STAGES - 1; ++n) fetch(n);
  float2 g[H] = {}, w[TAPS][H] = {}, rows[PAST + RW_N][H];   // the window, then the batch's rows
  if (on) {
    float v[RW_VEC];
    Vec<T, RW_VEC>::load(reinterpret_cast<const T*>(a.nw) + c, v);
#pragma unroll
    for (int i = 0; i < H; ++i) g[i] = make_float2(v[2 * i], v[2 * i + 1]);
    const T* conv = reinterpret_cast<const T*>(a.conv) + static_cast<long long>(c) * TAPS;
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < H; ++i)
        w[j][i] = make_float2(to_f(conv[2 * i * TAPS + j]) + (j == PAST ? 1.f : 0.f), to_f(conv[(2 * i + 1) * TAPS + j]) + (j == PAST ? 1.f : 0.f));
  }
#pragma unroll
  for (int k = 0; k < PAST; ++k)
#pragma unroll
    for (int i = 0; i < H; ++i) rows[k][i] = make_float2(0.f, 0.f);
  int b = rc_sequence(a, first), end = a.cu[b + 1];
  auto kept = [&](int k, int slot) {                 // row `slot` of what sequence b kept -> window row k
    const float* st = rc_past(a, b);
#pragma unroll
    for (int i = 0; i < H; ++i) rows[k][i] = on && st != nullptr ? *reinterpret_cast<const float2*>(st + static_cast<long long>(slot) * a.W + c + 2 * i) : make_float2(0.f, 0.f);
  };
  {  // a list that starts within PAST rows of a portion's start: what the sequence kept stands in front
    const int back = first - a.cu[b];
#pragma unroll
    for (int k = 0; k < PAST; ++k)
      if (back + k < PAST) kept(k, back + k);        // only looked at when the list starts with the portion
  }
  const int batches = (t1 - first + RW_N - 1) / RW_N;
  for (int n = 0; n < batches; ++n) {
    const int t = first + n * RW_N;
    asm volatile("cp.async.wait_group %0;" ::"n"(RW_STAGES - 2) : "memory");
    float ss[RW_N];
#pragma unroll
    for (int u = 0; u < RW_N; ++u) {
      const float4* src = reinterpret_cast<const float4*>(mine + (n % RW_STAGES * RW_N + u) * row);
      const float4 x = t + u < t1 ? src[0] : make_float4(0.f, 0.f, 0.f, 0.f), y = t + u < t1 ? src[1] : make_float4(0.f, 0.f, 0.f, 0.f);
      rows[PAST + u][0] = make_float2(x.x, x.y);
      rows[PAST + u][1] = make_float2(x.z, x.w);
      rows[PAST + u][2] = make_float2(y.x, y.y);
      rows[PAST + u][3] = make_float2(y.z, y.w);
      float2 q = mul2(rows[PAST + u][0], rows[PAST + u][0]);
#pragma unroll
      for (int i = 1; i < H; ++i) q = fma2(rows[PAST + u][i], rows[PAST + u][i], q);
      ss[u] = q.x + q.y;
    }
    if (n + RW_STAGES - 1 < batches) fetch(n + RW_STAGES - 1);   // into the stage that was read one batch ago
    else asm volatile("cp.async.commit_group;" ::: "memory");
    {  // four sums at once: after two steps a lane is in charge of one token
      const bool up16 = (lane & 16) != 0, up8 = (lane & 8) != 0;
      const float y0 = (up16 ? ss[2] : ss[0]) + __shfl_xor_sync(0xffffffffu, up16 ? ss[0] : ss[2], 16);
      const float y1 = (up16 ? ss[3] : ss[1]) + __shfl_xor_sync(0xffffffffu, up16 ? ss[1] : ss[3], 16);
      float y = (up8 ? y1 : y0) + __shfl_xor_sync(0xffffffffu, up8 ? y0 : y1, 8);
      y += __shfl_xor_sync(0xffffffffu, y, 4);
      y += __shfl_xor_sync(0xffffffffu, y, 2);
      y += __shfl_xor_sync(0xffffffffu, y, 1);
      if ((lane & 7) == 0) part[n & 1][warp][lane >> 3] = y;
    }
    __syncthreads();
    float sum[RW_N] = {};
    for (int k = 0; k < nw; ++k) {
      const float4 v = *reinterpret_cast<const float4*>(part[n & 1][k]);
      sum[0] += v.x; sum[1] += v.y; sum[2] += v.z; sum[3] += v.w;
    }
#pragma unroll
    for (int u = 0; u < RW_N; ++u) {
      const float r = rsqrtf(sum[u] / a.W + a.eps);
#pragma unroll
      for (int i = 0; i < H; ++i) rows[PAST + u][i] = mul2(mul2(rows[PAST + u][i], make_float2(r, r)), g[i]);
    }
    auto put = [&](int u, const float2 (&o)[H]) {
      if (!on || t + u < t0 || t + u >= t1) return;
      const float v[RW_VEC] = {o[0].x, o[0].y, o[1].x, o[1].y, o[2].x, o[2].y, o[3].x, o[3].y};
      Vec<T, RW_VEC>::store(reinterpret_cast<T*>(a.h) + static_cast<long long>(t + u) * a.W + c, v);
    };
    if (min(t + RW_N, t1) <= end) {                  // one portion (the same for the whole CTA)
#pragma unroll
      for (int u = 0; u < RW_N; ++u) {
        float2 o[H];
#pragma unroll
        for (int i = 0; i < H; ++i) {
          o[i] = mul2(w[PAST][i], rows[PAST + u][i]);
#pragma unroll
          for (int k = 0; k < PAST; ++k) o[i] = fma2(w[k][i], rows[u + k][i], o[i]);
        }
        put(u, o);
      }
#pragma unroll
      for (int k = 0; k < PAST; ++k)
#pragma unroll
        for (int i = 0; i < H; ++i) rows[k][i] = rows[RW_N + k][i];
    } else {
#pragma unroll
      for (int u = 0; u < RW_N; ++u) {
        if (t + u >= t1) break;
        if (t + u >= end) {                          // the next portion
          while (t + u >= end) { ++b; end = a.cu[b + 1]; }
#pragma unroll
          for (int k = 0; k < PAST; ++k) kept(k, k);
        }
        float2 o[H];
#pragma unroll
        for (int i = 0; i < H; ++i) {
          o[i] = mul2(w[PAST][i], rows[PAST + u][i]);
#pragma unroll
          for (int k = 0; k < PAST; ++k) o[i] = fma2(w[k][i], rows[k][i], o[i]);
        }
        put(u, o);
#pragma unroll
        for (int k = 0; k < PAST; ++k)
#pragma unroll
          for (int i = 0; i < H; ++i) rows[k][i] = k + 1 < PAST ? rows[k + 1 < PAST ? k + 1 : k][i] : rows[PAST + u][i];
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
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
rms_conv_state_kernel(const VbRmsConv a) {
  extern __shared__ float inv[];                     // [taps - 1]
  const int b = blockIdx.x, past = a.taps - 1, warp = threadIdx.x >> 5;
  const int s0 = a.cu[b], n = a.cu[b + 1] - s0;
  if (a.slots[b] < 0 || n <= 0) return;
  const bool zero = a.fresh != nullptr && a.fresh[b] != 0;
  for (int j = warp; j < past; j += 8) {
    const int at = n - past + j;
    const float f = at >= 0 ? rc_scale<VEC>(a.x + static_cast<long long>(s0 + at) * a.W, a.W, a.eps) : 0.f;
    if ((threadIdx.x & 31) == 0) inv[j] = f;
  }
  __syncthreads();
  float* st = a.state + static_cast<long long>(a.slots[b]) * a.slot_stride;
  for (int c = threadIdx.x * VEC; c < a.W; c += 256 * VEC) {
    float g[VEC], v[VEC];
    Vec<T, VEC>::load(reinterpret_cast<const T*>(a.nw) + c, g);
    for (int j = 0; j < past; ++j) {
      const int at = n - past + j;                   // reads ahead of what it writes
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
      if (at >= 0) {
        Vec<float, VEC>::load(a.x + static_cast<long long>(s0 + at) * a.W + c, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] *= inv[j] * g[i];
      } else if (!zero) {
        Vec<float, VEC>::load(st + static_cast<long long>(at + past) * a.W + c, v);
      }
      Vec<float, VEC>::store(st + static_cast<long long>(j) * a.W + c, v);
    }
  }
}

template <typename T, int VEC>
static int rms_conv_run(const VbRmsConv* p, cudaStream_t s) {
  const unsigned grid = static_cast<unsigned>((p->T + RC_RUN - 1) / RC_RUN);
  const int threads = ((p->W + VEC - 1) / VEC + 31) / 32 * 32;
  if (VEC == RW_VEC && threads <= 512 && p->taps <= 4) {
    const int smem = RW_STAGES * RW_N * threads * RW_VEC * 4;
    auto go = [&](auto kern) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
      kern<<<static_cast<unsigned>((p->T + RW_RUN - 1) / RW_RUN), threads, smem, s>>>(*p);
      return static_cast<int>(cudaGetLastError());
    };
    return p->taps == 1 ? go(rms_conv_once_kernel<T, 1>) : p->taps == 2 ? go(rms_conv_once_kernel<T, 2>) : p->taps == 3 ? go(rms_conv_once_kernel<T, 3>) : go(rms_conv_once_kernel<T, 4>);
  } else if (p->taps == 1) rms_conv_kernel<T, VEC, 1><<<grid, 256, 0, s>>>(*p);
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
    if (dtype == 0) vec ? rms_conv_state_kernel<float, 8><<<p->B, 256, p->taps * 4, s>>>(*p) : rms_conv_state_kernel<float, 1><<<p->B, 256, p->taps * 4, s>>>(*p);
    else vec ? rms_conv_state_kernel<bf16, 8><<<p->B, 256, p->taps * 4, s>>>(*p) : rms_conv_state_kernel<bf16, 1><<<p->B, 256, p->taps * 4, s>>>(*p);
    rc = static_cast<int>(cudaGetLastError());
  }
  return rc;
}
