// Preparation of grouped-query attention whose projections pass a short causal convolution over time: per row [q | k | v], the
// convolution of every channel, rotation of the query and key heads, an RMS norm without weight behind it, append to the paged
// cache, and the last inputs of the convolution kept per sequence (fp32). Compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>

namespace vb {

typedef __nv_bfloat16 bf16;

struct ConvUnit { int n, col, channel_row; bool is_q, is_v; };
__device__ __forceinline__ ConvUnit conv_unit(const VbConvPrep& a, int k) {
  ConvUnit u;
  u.is_q = k < a.H;
  u.is_v = k >= a.H + a.G;
  u.n = u.is_v ? a.vdim : a.dim;
  u.col = u.is_v ? (a.H + a.G) * a.dim + (k - a.H - a.G) * a.vdim : k * a.dim;
  u.channel_row = u.is_q ? 0 : (u.is_v ? a.G * a.dim + (k - a.H - a.G) * a.vdim : (k - a.H) * a.dim);   // place inside a cached row
  return u;
}
__device__ __forceinline__ int conv_sequence(const VbConvPrep& a, long long t) {
  int lo = 0, hi = a.B - 1;
  while (lo < hi) {
    const int mid = (lo + hi) / 2;
    if (a.cu[mid + 1] <= t) lo = mid + 1; else hi = mid;
  }
  return lo;
}
// The inputs in front of the portion (null: zeros).
__device__ __forceinline__ float* conv_past(const VbConvPrep& a, int b) {
  if (a.state == nullptr || a.slots == nullptr || a.slots[b] < 0 || (a.fresh != nullptr && a.fresh[b] != 0)) return nullptr;
  return a.state + static_cast<long long>(a.slots[b]) * a.slot_stride;
}

// A unit is one head row over a run of R tokens; L lanes share it, a lane holds eight consecutive channels of the unit (n <= 8 L)
// with their taps and the last inputs in registers.
template <typename T, int TAPS>
__global__ void __launch_bounds__(256)
conv_prep_kernel(const VbConvPrep a, int L, int R, long long units) {
  constexpr int VEC = 8, PAST = TAPS - 1;
  const long long u = (blockIdx.x * 256ll + threadIdx.x) / L;
  const int lane = threadIdx.x & (L - 1), per = a.H + 2 * a.G, C = (a.H + a.G) * a.dim + a.G * a.vdim;
  const bool live = u < units;
  const ConvUnit un = conv_unit(a, live ? static_cast<int>(u % per) : 0);
  const long long t0 = live ? u / per * R : 0;
  const int c = lane * VEC, k = live ? static_cast<int>(u % per) : 0;
  const bool in = live && c < un.n;
  const T* p = reinterpret_cast<const T*>(a.p);
  const int width = a.G * (a.dim + a.vdim);
  float w[VEC][TAPS], past[PAST > 0 ? PAST : 1][VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i)
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      w[i][j] = in && a.conv != nullptr ? to_f(reinterpret_cast<const T*>(a.conv)[static_cast<long long>(un.col + c + i) * TAPS + j]) : (j == TAPS - 1 ? 1.f : 0.f);
  int b = 0;
  long long s0 = 0, s1 = 0;
  // inputs of local tokens i - PAST .. i - 1
  auto refill = [&](long long t) {
    if constexpr (PAST > 0) {
      const float* st = nullptr;
      if (a.cu != nullptr) st = conv_past(a, b);
      else if (a.state != nullptr && a.active[t]) st = a.state + t * a.slot_stride;
      const long long i = a.cu != nullptr ? t - s0 : 0;
#pragma unroll
      for (int h = 0; h < PAST; ++h) {
        const long long at = i - PAST + h;
#pragma unroll
        for (int e = 0; e < VEC; ++e) past[h][e] = 0.f;
        if (!in) continue;
        if (at >= 0) Vec<T, VEC>::load(p + (s0 + at) * a.ldp + un.col + c, past[h]);
        else if (st != nullptr) Vec<float, VEC>::load(st + (at + PAST) * C + un.col + c, past[h]);
      }
    }
  };
  if (a.cu != nullptr && live) {
    b = conv_sequence(a, t0);
    s0 = a.cu[b];
    s1 = a.cu[b + 1];
  }
  if (live) refill(t0);
  for (int r = 0; r < R; ++r) {
    const long long t = t0 + r;
    const bool ok = live && t < a.T;
    float v[VEC], x[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = 0.f;
    if (ok && a.cu != nullptr && t >= s1) {
      while (b + 1 < a.B && t >= a.cu[b + 1]) ++b;
      s0 = a.cu[b];
      s1 = a.cu[b + 1];
      refill(t);
    }
    if (ok && in) Vec<T, VEC>::load(p + t * a.ldp + un.col + c, x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      v[i] = w[i][TAPS - 1] * x[i];
#pragma unroll
      for (int h = 0; h < PAST; ++h) v[i] += w[i][h] * past[h][i];
    }
    if constexpr (PAST > 0) {
#pragma unroll
      for (int h = 0; h + 1 < PAST; ++h)
#pragma unroll
        for (int i = 0; i < VEC; ++i) past[h][i] = past[h + 1][i];
#pragma unroll
      for (int i = 0; i < VEC; ++i) past[PAST - 1][i] = x[i];
      if (ok && in && a.cu == nullptr && a.state != nullptr && a.active[t]) {
#pragma unroll
        for (int h = 0; h < PAST; ++h) Vec<float, VEC>::store(a.state + t * a.slot_stride + h * C + un.col + c, past[h]);
      }
    }
    // rotation; the partner of (i, i + half) sits half / 8 lanes away
    const bool turn = ok && in && !un.is_v && c < 2 * a.half;
    const long long tab = turn ? static_cast<long long>(min(max(a.pos[t], 0), a.max_pos - 1)) * a.half : 0;
    if (a.halves) {
      const int off = a.half / VEC, first = c < a.half;
      const int src = c < 2 * a.half ? (first ? lane + off : lane - off) : lane;
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float o = __shfl_sync(0xffffffffu, v[i], src, L);
        if (turn) {
          const int f = (first ? c : c - a.half) + i;
          const float cs = a.cos_t[tab + f], sn = a.sin_t[tab + f];
          v[i] = first ? v[i] * cs - o * sn : v[i] * cs + o * sn;
        }
      }
    } else if (turn) {
#pragma unroll
      for (int i = 0; i < VEC; i += 2)
        if (c + i < 2 * a.half) {
          const float cs = a.cos_t[tab + ((c + i) >> 1)], sn = a.sin_t[tab + ((c + i) >> 1)], y = v[i], z = v[i + 1];
          v[i] = y * cs - z * sn;
          v[i + 1] = z * cs + y * sn;
        }
    }
    float ss = 0.f;
    if (!un.is_v) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += v[i] * v[i];
    }
    for (int s = L >> 1; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    if (!ok || !in) continue;
    if (!un.is_v) {
      const float f = 1.f / sqrtf(ss / un.n + a.eps);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] *= f;
    }
    if (un.is_q) {
      Vec<T, VEC>::store(reinterpret_cast<T*>(a.q) + (t * a.H + k) * a.dim + c, v);
    } else {
      if (a.rows != nullptr) Vec<T, VEC>::store(reinterpret_cast<T*>(a.rows) + t * a.ldr + un.channel_row + c, v);
      if (a.pages != nullptr) {
        const long long sl = a.page_slot[t];
        if (sl >= 0 && sl < a.num_slots)
          Vec<T, VEC>::store(reinterpret_cast<T*>(a.pages) + (sl / a.block_size) * a.page_stride + (sl % a.block_size) * width + un.channel_row + c, v);
      }
    }
  }
}

// Any sizes and any number of taps: one warp per head row of a token, the row staged in shared memory.
template <typename T>
__global__ void __launch_bounds__(128)
conv_prep_any_kernel(const VbConvPrep a, long long units) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, per = a.H + 2 * a.G, C = (a.H + a.G) * a.dim + a.G * a.vdim, past = a.taps - 1;
  const long long u = blockIdx.x * 4ll + warp;
  if (u >= units) return;
  float* row = sm + warp * max(a.dim, a.vdim);
  const int k = static_cast<int>(u % per);
  const long long t = u / per;
  const ConvUnit un = conv_unit(a, k);
  const T *p = reinterpret_cast<const T*>(a.p), *conv = reinterpret_cast<const T*>(a.conv);
  long long s0 = t;                      // steps: every token is the first of its portion
  float* st = nullptr;
  if (a.cu != nullptr) {
    const int b = conv_sequence(a, t);
    s0 = a.cu[b];
    st = conv_past(a, b);
  } else if (a.state != nullptr && a.active[t]) {
    st = a.state + t * a.slot_stride;
  }
  float ss = 0.f;
  for (int c = lane; c < un.n; c += 32) {
    float v = 0.f;
    if (conv == nullptr) {
      v = to_f(p[t * a.ldp + un.col + c]);
    } else {
      for (int j = 0; j < a.taps; ++j) {
        const long long at = t - s0 - past + j;
        const float x = at >= 0 ? to_f(p[(s0 + at) * a.ldp + un.col + c]) : (st != nullptr ? st[(at + past) * C + un.col + c] : 0.f);
        v += to_f(conv[static_cast<long long>(un.col + c) * a.taps + j]) * x;
      }
    }
    row[c] = v;
    if (a.cu == nullptr && st != nullptr && past > 0) {
      for (int j = 0; j + 1 < past; ++j) st[j * C + un.col + c] = st[(j + 1) * C + un.col + c];
      st[(past - 1) * C + un.col + c] = to_f(p[t * a.ldp + un.col + c]);
    }
  }
  __syncwarp();
  const long long tab = static_cast<long long>(min(max(a.pos[t], 0), a.max_pos - 1)) * a.half;
  auto turned = [&](int c) {
    if (un.is_v || c >= 2 * a.half) return row[c];
    const int f = a.halves ? (c < a.half ? c : c - a.half) : c >> 1;
    const bool first = a.halves ? c < a.half : (c & 1) == 0;
    const float o = row[a.halves ? (first ? c + a.half : c - a.half) : c ^ 1], cs = a.cos_t[tab + f], sn = a.sin_t[tab + f];
    return first ? row[c] * cs - o * sn : row[c] * cs + o * sn;
  };
  for (int c = lane; c < un.n; c += 32) {
    const float v = turned(c);
    ss += v * v;
  }
  const float f = un.is_v ? 1.f : 1.f / sqrtf(warp_sum(ss) / un.n + a.eps);
  T *d0 = nullptr, *d1 = nullptr;
  if (un.is_q) {
    d0 = reinterpret_cast<T*>(a.q) + (t * a.H + k) * a.dim;
  } else {
    if (a.rows != nullptr) d0 = reinterpret_cast<T*>(a.rows) + t * a.ldr + un.channel_row;
    if (a.pages != nullptr) {
      const long long sl = a.page_slot[t];
      if (sl >= 0 && sl < a.num_slots)
        d1 = reinterpret_cast<T*>(a.pages) + (sl / a.block_size) * a.page_stride + (sl % a.block_size) * (a.G * (a.dim + a.vdim)) + un.channel_row;
    }
  }
  for (int c = lane; c < un.n; c += 32) {
    const float v = turned(c) * f;
    if (d0 != nullptr) d0[c] = from_f<T>(v);
    if (d1 != nullptr) d1[c] = from_f<T>(v);
  }
}

// The last taps - 1 inputs of every portion (a portion shorter than that moves older ones up).
template <typename T>
__global__ void conv_state_kernel(const VbConvPrep a, int C) {
  const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x, past = a.taps - 1;
  if (c >= C || a.slots[b] < 0) return;
  const long long s0 = a.cu[b], n = a.cu[b + 1] - s0;
  if (n <= 0) return;
  const bool zero = a.fresh != nullptr && a.fresh[b] != 0;
  float* st = a.state + static_cast<long long>(a.slots[b]) * a.slot_stride + c;
  for (int j = 0; j < past; ++j) {
    const long long at = n - past + j;   // reads ahead of what it writes
    st[static_cast<long long>(j) * C] = at >= 0 ? to_f(reinterpret_cast<const T*>(a.p)[(s0 + at) * a.ldp + c]) : (zero ? 0.f : st[(at + past) * C]);
  }
}

}  // namespace vb

using namespace vb;

extern "C" int vb_conv_prep(int dtype, const VbConvPrep* p, cudaStream_t s) {
  if (p->T <= 0) return 0;
  auto mis = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) != 0; };
  const int C = (p->H + p->G) * p->dim + p->G * p->vdim, per = p->H + 2 * p->G, most = p->dim > p->vdim ? p->dim : p->vdim;
  const bool vec = p->dim % 8 == 0 && p->vdim % 8 == 0 && most <= 256 && p->taps <= 4 && p->ldp % 8 == 0 && p->ldr % 8 == 0 && p->page_stride % 8 == 0 &&
                   p->slot_stride % 4 == 0 && (!p->halves || p->half % 8 == 0) && !mis(p->p) && !mis(p->q) && !mis(p->rows) && !mis(p->pages) && !mis(p->state);
  if (p->B > 65535) return -1;
  if (vec) {
    int L = 1;
    while (L < 32 && L * 8 < most) L *= 2;
    // long runs reuse the inputs, short ones fill the GPU
    const int R = p->cu == nullptr ? 1 : (static_cast<long long>(p->T) * per * L > 148ll * 2048 * 32 ? 16 : 4);
    const long long units = (p->T + R - 1ll) / R * per;
    const unsigned grid = static_cast<unsigned>((units * L + 255) / 256);
    auto go = [&](auto kern) { kern<<<grid, 256, 0, s>>>(*p, L, R, units); };
    if (dtype == 0) {
      if (p->taps == 1) go(conv_prep_kernel<float, 1>);
      else if (p->taps == 2) go(conv_prep_kernel<float, 2>);
      else if (p->taps == 3) go(conv_prep_kernel<float, 3>);
      else go(conv_prep_kernel<float, 4>);
    } else {
      if (p->taps == 1) go(conv_prep_kernel<bf16, 1>);
      else if (p->taps == 2) go(conv_prep_kernel<bf16, 2>);
      else if (p->taps == 3) go(conv_prep_kernel<bf16, 3>);
      else go(conv_prep_kernel<bf16, 4>);
    }
  } else {
    const long long units = static_cast<long long>(p->T) * per;
    const unsigned grid = static_cast<unsigned>((units + 3) / 4);
    const int smem = 4 * most * 4;
    if (smem > 48 * 1024) return -2;
    if (dtype == 0) conv_prep_any_kernel<float><<<grid, 128, smem, s>>>(*p, units);
    else conv_prep_any_kernel<bf16><<<grid, 128, smem, s>>>(*p, units);
  }
  if (p->cu != nullptr && p->state != nullptr && p->slots != nullptr && p->taps > 1) {
    const dim3 grid((C + 255) / 256, p->B);
    if (dtype == 0) conv_state_kernel<float><<<grid, 256, 0, s>>>(*p, C);
    else conv_state_kernel<bf16><<<grid, 256, 0, s>>>(*p, C);
  }
  return static_cast<int>(cudaGetLastError());
}
