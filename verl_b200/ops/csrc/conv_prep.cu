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
  u.is_v = k >= a.H + a.G;       // a.GV heads
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

// Eight consecutive elements as loaded; unpacking is left to the place of use, so that all loads go out first.
template <typename T> struct Raw8;
template <> struct Raw8<bf16> {
  uint4 a;
  __device__ __forceinline__ void load(const bf16* p) { a = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void zero() { a = make_uint4(0, 0, 0, 0); }
  __device__ __forceinline__ void get(float (&v)[8]) const {
    const uint32_t u[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[2 * i] = __uint_as_float(u[i] << 16);
      v[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    }
  }
};
template <> struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) { a = reinterpret_cast<const float4*>(p)[0]; b = reinterpret_cast<const float4*>(p)[1]; }
  __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void get(float (&v)[8]) const {
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
};

// L lanes share a head row, a lane holds eight consecutive channels (n <= 8 L) of N consecutive tokens: taps and the window of inputs
// stay in registers. A block takes one head.
template <typename T, int TAPS, int N>
__global__ void __launch_bounds__(256, 2)
conv_prep_kernel(const VbConvPrep a, int L) {
  constexpr int VEC = 8, PAST = TAPS - 1;
  const int lane = threadIdx.x & (L - 1), k = blockIdx.y, C = (a.H + a.G) * a.dim + a.GV * a.vdim, c = lane * VEC;
  const int t0 = (blockIdx.x * (256 / L) + threadIdx.x / L) * N;
  const ConvUnit un = conv_unit(a, k);
  const bool mine = c < un.n && t0 < a.T, rot = !un.is_v && c < 2 * a.half;
  const T* p = reinterpret_cast<const T*>(a.p) + static_cast<long long>(t0) * a.ldp + un.col + c;
  Raw8<T> raw[N];
  int where[N];
#pragma unroll
  for (int u = 0; u < N; ++u) {
    if (mine && t0 + u < a.T) raw[u].load(p + u * a.ldp);
    else raw[u].zero();
    where[u] = rot && t0 + u < a.T ? min(max(a.pos[t0 + u], 0), a.max_pos - 1) : 0;
  }
  float w[VEC * TAPS], past[PAST > 0 ? PAST : 1][VEC];
  if (a.conv != nullptr && mine) {       // the lane's taps are consecutive: [channel, tap]
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      Vec<T, VEC>::load(reinterpret_cast<const T*>(a.conv) + static_cast<long long>(un.col + c) * TAPS + j * VEC, *reinterpret_cast<float(*)[VEC]>(w + j * VEC));
  } else {
#pragma unroll
    for (int i = 0; i < VEC * TAPS; ++i) w[i] = i % TAPS == PAST ? 1.f : 0.f;
  }
  // the inputs in front of token t: rows of its portion, then what the sequence kept, then zeros
  int s1 = 0;                            // end of the portion
  float* st = nullptr;
  auto refill = [&](int t) {
    int back = 0;
    if (a.cu != nullptr) {
      const int b = conv_sequence(a, t);
      back = t - a.cu[b];
      s1 = a.cu[b + 1];
      st = back < PAST ? conv_past(a, b) : nullptr;
    } else {
      s1 = t + 1;
      st = a.state != nullptr && a.active[t] ? a.state + static_cast<long long>(t) * a.slot_stride : nullptr;
    }
#pragma unroll
    for (int h = 0; h < PAST; ++h) {
      const int at = back - PAST + h;    // index inside the portion
#pragma unroll
      for (int i = 0; i < VEC; ++i) past[h][i] = 0.f;
      if (at >= 0) Vec<T, VEC>::load(p + static_cast<long long>(t - t0 - PAST + h) * a.ldp, past[h]);
      else if (st != nullptr) Vec<float, VEC>::load(st + static_cast<long long>(at + PAST) * C + un.col + c, past[h]);
    }
  };
  if (PAST > 0 && mine) refill(t0);
  const bool first = c < a.half;         // of a pair of halves
  const int src = a.halves && c < 2 * a.half ? (first ? lane + a.half / VEC : lane - a.half / VEC) : lane;
  const float inv_n = 1.f / un.n;
#pragma unroll
  for (int u = 0; u < N; ++u) {
    const int t = t0 + u;
    const bool ok = mine && t < a.T;
    float cs[VEC], sn[VEC], x[VEC], v[VEC];
    if (rot && ok) {
      const long long tab = static_cast<long long>(where[u]) * a.half;
      if (a.halves) {
        Vec<float, VEC>::load(a.cos_t + tab + (first ? c : c - a.half), cs);
        Vec<float, VEC>::load(a.sin_t + tab + (first ? c : c - a.half), sn);
      } else {
#pragma unroll
        for (int i = 0; i < VEC; i += 2) {
          cs[i] = c + i < 2 * a.half ? a.cos_t[tab + ((c + i) >> 1)] : 1.f;
          sn[i] = c + i < 2 * a.half ? a.sin_t[tab + ((c + i) >> 1)] : 0.f;
        }
      }
    }
    raw[u].get(x);
    if (PAST > 0 && u > 0 && ok && t >= s1) refill(t);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      v[i] = w[i * TAPS + PAST] * x[i];
#pragma unroll
      for (int h = 0; h < PAST; ++h) v[i] += w[i * TAPS + h] * past[h][i];
    }
    if constexpr (PAST > 0) {
#pragma unroll
      for (int h = 0; h + 1 < PAST; ++h)
#pragma unroll
        for (int i = 0; i < VEC; ++i) past[h][i] = past[h + 1][i];
#pragma unroll
      for (int i = 0; i < VEC; ++i) past[PAST - 1][i] = x[i];
      if (N == 1 && ok && a.cu == nullptr && st != nullptr) {   // a step keeps its inputs itself
#pragma unroll
        for (int h = 0; h < PAST; ++h) Vec<float, VEC>::store(st + static_cast<long long>(h) * C + un.col + c, past[h]);
      }
    }
    if (!un.is_v && (a.half > 0 || a.norm)) {   // the same for the whole block
      // rotation; the partner of (i, i + half) sits half / 8 lanes away
      if (a.halves) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const float o = __shfl_sync(0xffffffffu, v[i], src, L);
          if (rot && ok) v[i] = v[i] * cs[i] + (first ? -o : o) * sn[i];
        }
      } else if (rot && ok) {
#pragma unroll
        for (int i = 0; i < VEC; i += 2) {
          const float y = v[i], z = v[i + 1];
          v[i] = y * cs[i] - z * sn[i];
          v[i + 1] = z * cs[i] + y * sn[i];
        }
      }
      if (a.norm) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss += v[i] * v[i];
        if (c >= un.n) ss = 0.f;
        for (int m = L >> 1; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
        const float f = rsqrtf(ss * inv_n + a.eps);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] *= f;
      }
    }
    if (!ok) continue;
    if (un.is_q) {
      Vec<T, VEC>::store(reinterpret_cast<T*>(a.q) + (static_cast<long long>(t) * a.H + k) * a.dim + c, v);
    } else {
      if (a.rows != nullptr) Vec<T, VEC>::store(reinterpret_cast<T*>(a.rows) + t * a.ldr + un.channel_row + c, v);
      if (a.pages != nullptr) {
        const long long sl = a.page_slot[t];
        if (sl >= 0 && sl < a.num_slots) {
          const unsigned blk = static_cast<unsigned>(sl) / static_cast<unsigned>(a.block_size), at = static_cast<unsigned>(sl) - blk * a.block_size;
          Vec<T, VEC>::store(reinterpret_cast<T*>(a.pages) + blk * a.page_stride + static_cast<long long>(at) * (a.G * a.dim + a.GV * a.vdim) + un.channel_row + c, v);
        }
      }
    }
  }
}

// Any sizes and any number of taps: one warp per head row of a token, the row staged in shared memory.
template <typename T>
__global__ void __launch_bounds__(128)
conv_prep_any_kernel(const VbConvPrep a, long long units) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, per = a.H + a.G + a.GV, C = (a.H + a.G) * a.dim + a.GV * a.vdim, past = a.taps - 1;
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
  const float f = un.is_v || !a.norm ? 1.f : 1.f / sqrtf(warp_sum(ss) / un.n + a.eps);
  T *d0 = nullptr, *d1 = nullptr;
  if (un.is_q) {
    d0 = reinterpret_cast<T*>(a.q) + (t * a.H + k) * a.dim;
  } else {
    if (a.rows != nullptr) d0 = reinterpret_cast<T*>(a.rows) + t * a.ldr + un.channel_row;
    if (a.pages != nullptr) {
      const long long sl = a.page_slot[t];
      if (sl >= 0 && sl < a.num_slots)
        d1 = reinterpret_cast<T*>(a.pages) + (sl / a.block_size) * a.page_stride + (sl % a.block_size) * (a.G * a.dim + a.GV * a.vdim) + un.channel_row;
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
  const int C = (p->H + p->G) * p->dim + p->GV * p->vdim, per = p->H + p->G + p->GV, most = p->dim > p->vdim ? p->dim : p->vdim;
  const bool vec = p->num_slots < (1ll << 31) && per <= 65535 && p->dim % 8 == 0 && p->vdim % 8 == 0 && most <= 256 && p->taps <= 4 && p->ldp % 8 == 0 && p->ldr % 8 == 0 && p->page_stride % 8 == 0 &&
                   p->slot_stride % 4 == 0 && (!p->halves || p->half % 8 == 0) && !mis(p->p) && !mis(p->q) && !mis(p->rows) && !mis(p->pages) && !mis(p->state) &&
                   !mis(p->cos_t) && !mis(p->sin_t) && !mis(p->conv);
  if (p->B > 65535) return -1;
  if (vec) {
    int L = 1;
    while (L < 32 && L * 8 < most) L *= 2;
    const int n = p->cu != nullptr && static_cast<long long>(p->T) * per * L >= 148ll * 512 * 4 ? 4 : 1;     // tokens per thread
    const dim3 grid((p->T + 256 / L * n - 1) / (256 / L * n), per);
    auto go = [&](auto kern) { kern<<<grid, 256, 0, s>>>(*p, L); };
#define VB_CONV(T_, N_)                                                                              \
  (p->taps == 1 ? go(conv_prep_kernel<T_, 1, N_>) : p->taps == 2 ? go(conv_prep_kernel<T_, 2, N_>)   \
   : p->taps == 3 ? go(conv_prep_kernel<T_, 3, N_>) : go(conv_prep_kernel<T_, 4, N_>))
    if (n == 4) dtype == 0 ? VB_CONV(float, 4) : VB_CONV(bf16, 4);
    else dtype == 0 ? VB_CONV(float, 1) : VB_CONV(bf16, 1);
#undef VB_CONV
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
