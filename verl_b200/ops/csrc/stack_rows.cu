// Row kernels of stacks with norms on the sublayers' outputs: normed embedding, residual add of a normed sublayer output (which
// also adds up split-K partial products and the rows of chosen experts; RMS or Dynamic Tanh), gated activations, gated RMS norm
// of a row or of its heads, and the preparation of grouped-query attention (norm and rotation of query and key heads, or norms over whole
// projections, value mixing, append to the paged cache), and the normed difference of two attention maps.
// Statistics, angles and the residual stream are fp32; compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>
#include <type_traits>

namespace vb {

typedef __nv_bfloat16 bf16;

// --------------------------------------------------------------------------------------------- embedding + RMS norm
template <typename T, int VEC>
__global__ void embed_rms_kernel(const long long* __restrict__ ids, const T* __restrict__ w, float scale, const T* __restrict__ nw, float eps,
                                 float* __restrict__ x, T* __restrict__ h, int W, int V) {
  __shared__ float red[33];
  const long long t = blockIdx.x, id = ids[t];
  const bool ok = id >= 0 && id < V;
  const T* row = w + (ok ? id : 0) * W;
  float v[VEC], g[VEC], ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    Vec<T, VEC>::load(row + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += v[i] * scale * (v[i] * scale);
  }
  const float r = ok ? 1.f / sqrtf(block_sum(ss, red) / W + eps) : 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    Vec<T, VEC>::load(row + c, v);
    Vec<T, VEC>::load(nw + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * scale * r * g[i];
    Vec<float, VEC>::store(x + t * W + c, v);
    Vec<T, VEC>::store(h + t * W + c, v);
  }
}

// --------------------------------------------------------------------------------------------- residual + RMS norm
// One CTA per token; a thread keeps its ITEMS x VEC columns of the sublayer output in registers between the two passes.
template <typename T, int VEC, int ITEMS>
__global__ void residual_rms_kernel(const VbResidRms p) {
  __shared__ float red[33];
  const long long t = blockIdx.x;
  float y[ITEMS][VEC], v[VEC];
  float* xr = p.x + t * p.W;
  const T* rows = reinterpret_cast<const T*>(p.rows);
  const float gate = p.gate != nullptr ? sigmoid_f(p.gate[t * p.ldgate]) : 1.f;
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
#pragma unroll
    for (int i = 0; i < VEC; ++i) y[it][i] = 0.f;
    if (c >= p.W) continue;
    if (p.y != nullptr) {
      if (p.y_f32) {
        const float* src = reinterpret_cast<const float*>(p.y) + t * p.ldy + c;
        for (int s = 0; s < p.splits; ++s) {
          Vec<float, VEC>::load(src + s * p.split_stride, v);
#pragma unroll
          for (int i = 0; i < VEC; ++i) y[it][i] += v[i];
        }
      } else {
        Vec<T, VEC>::load(reinterpret_cast<const T*>(p.y) + t * p.ldy + c, y[it]);
      }
      if (p.gate != nullptr) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[it][i] *= gate;
      }
    }
    if (rows != nullptr) {
      for (int j = 0; j < p.top; ++j) {
        Vec<T, VEC>::load(rows + static_cast<long long>(p.slot[t * p.top + j]) * p.ldr + c, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[it][i] += v[i];
      }
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += y[it][i] * y[it][i];
  }
  const float r = p.mult / sqrtf(block_sum(ss, red) / p.W + p.eps);
  const T *nw = reinterpret_cast<const T*>(p.nw), *next = reinterpret_cast<const T*>(p.next);
  T* hr = reinterpret_cast<T*>(p.h) + t * p.W;
  ss = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
    if (c >= p.W) continue;
    float x[VEC];
    Vec<float, VEC>::load(xr + c, x);
    Vec<T, VEC>::load(nw + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      x[i] += y[it][i] * r * v[i];
      y[it][i] = x[i];
      ss += x[i] * x[i];
    }
    Vec<float, VEC>::store(xr + c, x);
    if (next == nullptr) Vec<T, VEC>::store(hr + c, x);
  }
  if (next == nullptr) return;
  const float rn = 1.f / sqrtf(block_sum(ss, red) / p.W + p.eps);
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
    if (c >= p.W) continue;
    Vec<T, VEC>::load(next + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) y[it][i] *= rn * v[i];
    Vec<T, VEC>::store(hr + c, y[it]);
  }
}

template <typename T, int VEC>
static int residual_rms(const VbResidRms* p, cudaStream_t s) {
  const int nvec = (p->W + VEC - 1) / VEC;
  int thr = nvec >= 256 ? 256 : (nvec + 31) / 32 * 32;
  if (nvec > 8 * thr) thr = 1024;
  const int items = (nvec + thr - 1) / thr;
  auto go = [&](auto kern) {
    kern<<<p->T, thr, 0, s>>>(*p);
    return static_cast<int>(cudaGetLastError());
  };
  if (items == 1) return go(residual_rms_kernel<T, VEC, 1>);
  if (items == 2) return go(residual_rms_kernel<T, VEC, 2>);
  if (items <= 4) return go(residual_rms_kernel<T, VEC, 4>);
  if (items <= 8) return go(residual_rms_kernel<T, VEC, 8>);
  return -1;
}

// --------------------------------------------------------------------------------------------- residual + Dynamic Tanh of experts' rows
// Elementwise: a thread owns VEC columns of one token, requests all its rows before it uses the first.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) residual_dyt_kernel(const VbResidDyt p, long long total) {
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= total) return;
  const int per = p.W / VEC, c = static_cast<int>(i % per) * VEC;
  const long long t = i / per;
  const T* rows = reinterpret_cast<const T*>(p.rows);
  const int* slot = p.slot + t * p.top;
  float x[VEC], y[VEC], v[4][VEC], w[VEC], b[VEC];
  Vec<float, VEC>::load(p.x + t * p.W + c, x);
#pragma unroll
  for (int k = 0; k < VEC; ++k) y[k] = 0.f;
  for (int j = 0; j < p.top; j += 4) {
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (j + u < p.top) Vec<T, VEC>::load(rows + static_cast<long long>(slot[j + u]) * p.ldr + c, v[u]);
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (j + u < p.top) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) y[k] += v[u][k];
      }
  }
  const float pa = to_f(*reinterpret_cast<const T*>(p.palpha)), na = to_f(*reinterpret_cast<const T*>(p.alpha));
  Vec<T, VEC>::load(reinterpret_cast<const T*>(p.pw) + c, w);
  Vec<T, VEC>::load(reinterpret_cast<const T*>(p.pb) + c, b);
#pragma unroll
  for (int k = 0; k < VEC; ++k) x[k] += tanhf(pa * y[k]) * w[k] + b[k];
  Vec<float, VEC>::store(p.x + t * p.W + c, x);
  Vec<T, VEC>::load(reinterpret_cast<const T*>(p.nw) + c, w);
  Vec<T, VEC>::load(reinterpret_cast<const T*>(p.nb) + c, b);
#pragma unroll
  for (int k = 0; k < VEC; ++k) x[k] = tanhf(na * x[k]) * w[k] + b[k];
  Vec<T, VEC>::store(reinterpret_cast<T*>(p.h) + t * p.W + c, x);
}

// --------------------------------------------------------------------------------------------- rms_norm(o) * w * sigmoid(g) over whole rows
template <typename T, int VEC, int ITEMS>
__global__ void gated_rms_kernel(const T* __restrict__ o, long long ldo, const T* __restrict__ g, long long ldg, const T* __restrict__ norm, float eps,
                                 T* __restrict__ out, int W) {
  __shared__ float red[33];
  const long long t = blockIdx.x;
  float v[ITEMS][VEC], z[ITEMS][VEC], w[VEC], ss = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
    if (c >= W) continue;
    Vec<T, VEC>::load(o + t * ldo + c, v[it]);
    Vec<T, VEC>::load(g + t * ldg + c, z[it]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss += v[it][k] * v[it][k];
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / W + eps);
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * blockDim.x + threadIdx.x) * VEC;
    if (c >= W) continue;
    Vec<T, VEC>::load(norm + c, w);
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[it][k] = v[it][k] * r * w[k] * sigmoid_f(z[it][k]);
    Vec<T, VEC>::store(out + t * W + c, v[it]);
  }
}

template <typename T, int VEC>
static int gated_rms(const void* o, long long ldo, const void* g, long long ldg, const void* norm, float eps, void* out, int T_, int W, cudaStream_t s) {
  const int nvec = (W + VEC - 1) / VEC;
  int thr = nvec >= 256 ? 256 : (nvec + 31) / 32 * 32;
  if (nvec > 8 * thr) thr = 1024;
  const int items = (nvec + thr - 1) / thr;
  auto go = [&](auto kern) {
    kern<<<T_, thr, 0, s>>>((const T*)o, ldo, (const T*)g, ldg, (const T*)norm, eps, (T*)out, W);
    return static_cast<int>(cudaGetLastError());
  };
  if (items == 1) return go(gated_rms_kernel<T, VEC, 1>);
  if (items == 2) return go(gated_rms_kernel<T, VEC, 2>);
  if (items <= 4) return go(gated_rms_kernel<T, VEC, 4>);
  if (items <= 8) return go(gated_rms_kernel<T, VEC, 8>);
  if (VEC == 1 && items <= 32) return go(gated_rms_kernel<T, VEC, 32>);
  return -1;
}

// --------------------------------------------------------------------------------------------- the same with one norm per head
// L lanes share a head row of one token (n <= 32 VEC ITEMS columns).
template <typename T, int VEC, int ITEMS>
__global__ void __launch_bounds__(256)
gated_rms_heads_kernel(const T* __restrict__ o, long long ldo, const T* __restrict__ g, long long ldg, const T* __restrict__ norm, float eps, T* __restrict__ out,
                       int n, int heads, int L, long long units) {
  const long long u = (blockIdx.x * 256ll + threadIdx.x) / L;
  const int lane = threadIdx.x & (L - 1);
  const bool live = u < units;
  const long long t = live ? u / heads : 0;
  const int col = live ? static_cast<int>(u % heads) * n : 0;
  float v[ITEMS][VEC], z[ITEMS][VEC], w[VEC], ss = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * L + lane) * VEC;
    if (!live || c >= n) continue;
    Vec<T, VEC>::load(o + t * ldo + col + c, v[it]);
    Vec<T, VEC>::load(g + t * ldg + col + c, z[it]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss += v[it][k] * v[it][k];
  }
  for (int m = L >> 1; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  const float r = 1.f / sqrtf(ss / n + eps);
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int c = (it * L + lane) * VEC;
    if (!live || c >= n) continue;
    Vec<T, VEC>::load(norm + col + c, w);
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[it][k] = v[it][k] * r * w[k] * sigmoid_f(z[it][k]);
    Vec<T, VEC>::store(out + t * (static_cast<long long>(heads) * n) + col + c, v[it]);
  }
}

template <typename T, int VEC>
static int gated_rms_heads(const void* o, long long ldo, const void* g, long long ldg, const void* norm, float eps, void* out, int T_, int n, int heads, cudaStream_t s) {
  int L = 1;
  while (L < 32 && L * VEC < n) L *= 2;
  const int items = (n + L * VEC - 1) / (L * VEC);
  const long long units = static_cast<long long>(T_) * heads;
  auto go = [&](auto kern) {
    kern<<<static_cast<unsigned>((units * L + 255) / 256), 256, 0, s>>>((const T*)o, ldo, (const T*)g, ldg, (const T*)norm, eps, (T*)out, n, heads, L, units);
    return static_cast<int>(cudaGetLastError());
  };
  if (items == 1) return go(gated_rms_heads_kernel<T, VEC, 1>);
  if (items <= 4) return go(gated_rms_heads_kernel<T, VEC, 4>);
  if (items <= 16) return go(gated_rms_heads_kernel<T, VEC, 16>);
  return -1;
}

// --------------------------------------------------------------------------------------------- difference of two attention maps
// One warp per (token, head): a [T, 2 H, dv] -> (1 - diff) rms_norm(a0 - lambda a1).
template <typename A, typename T>
__global__ void __launch_bounds__(128)
diff_combine_kernel(const A* __restrict__ a, const T* __restrict__ vec, int dim, float diff, float eps, T* __restrict__ out, long long rows, int dv) {
  const int lane = threadIdx.x & 31;
  const long long u = blockIdx.x * 4ll + (threadIdx.x >> 5);
  if (u >= rows) return;
  float x = 0.f, y = 0.f;
  for (int i = lane; i < dim; i += 32) {
    x += to_f(vec[i]) * to_f(vec[dim + i]);
    y += to_f(vec[2 * dim + i]) * to_f(vec[3 * dim + i]);
  }
  const float lam = expf(warp_sum(x)) - expf(warp_sum(y)) + diff;
  const A *a0 = a + 2 * u * dv, *a1 = a0 + dv;
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) {
    const float z = to_f(a0[c]) - lam * to_f(a1[c]);
    ss += z * z;
  }
  const float r = (1.f - diff) / sqrtf(warp_sum(ss) / dv + eps);
  for (int c = lane; c < dv; c += 32) out[u * dv + c] = from_f<T>((to_f(a0[c]) - lam * to_f(a1[c])) * r);
}

// --------------------------------------------------------------------------------------------- norms over whole query and key projections
// One CTA per token.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
whole_norm_kernel(const VbWholeNorm a) {
  __shared__ float red[33];
  const long long t = blockIdx.x;
  const int nq = a.H * a.dim, nk = a.G * a.dim, nv = a.G * a.vdim;
  const T* p = reinterpret_cast<const T*>(a.p) + t * a.ldp;
  float v[VEC], w[VEC], sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * VEC; c < nq + nk; c += 256 * VEC) {
    Vec<T, VEC>::load(p + c, v);
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) s += v[i] * v[i];
    if (c < nq) sq += s; else sk += s;
  }
  const float rq = 1.f / sqrtf(block_sum(sq, red) / nq + a.eps), rk = 1.f / sqrtf(block_sum(sk, red) / nk + a.eps);
  T* q = reinterpret_cast<T*>(a.q) + t * nq;
  T* d0 = a.rows != nullptr ? reinterpret_cast<T*>(a.rows) + t * a.ldr : nullptr;
  T* d1 = nullptr;
  if (a.pages != nullptr) {
    const long long sl = a.page_slot[t];
    if (sl >= 0 && sl < a.num_slots) d1 = reinterpret_cast<T*>(a.pages) + (sl / a.block_size) * a.page_stride + (sl % a.block_size) * (nk + nv);
  }
  for (int c = threadIdx.x * VEC; c < nq + nk + nv; c += 256 * VEC) {
    Vec<T, VEC>::load(p + c, v);
    if (c < nq) {
      const float f = rq * to_f(reinterpret_cast<const T*>(a.temp)[c / a.dim]);
      Vec<T, VEC>::load(reinterpret_cast<const T*>(a.qn) + c, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = v[i] * f * w[i];
      Vec<T, VEC>::store(q + c, v);
      continue;
    }
    const int at = c - nq;
    if (at < nk) {
      Vec<T, VEC>::load(reinterpret_cast<const T*>(a.kn) + at, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = v[i] * rk * w[i];
    }
    if (d0 != nullptr) Vec<T, VEC>::store(d0 + at, v);
    if (d1 != nullptr) Vec<T, VEC>::store(d1 + at, v);
  }
}

// --------------------------------------------------------------------------------------------- silu(r g) * (r u), or the clipped form
template <typename T, int VEC>
__global__ void gated_silu_kernel(const T* __restrict__ gu, long long ldg, const float* __restrict__ row_scale, float clip, T* __restrict__ out, int I,
                                  long long total) {
  const long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x;
  if (i >= total) return;
  const int per = I / VEC, c = static_cast<int>(i % per) * VEC;
  const long long t = i / per;
  const float r = row_scale != nullptr ? row_scale[t] : 1.f;
  float g[VEC], u[VEC];
  Vec<T, VEC>::load(gu + t * ldg + c, g);
  Vec<T, VEC>::load(gu + t * ldg + I + c, u);
#pragma unroll
  for (int k = 0; k < VEC; ++k) {
    if (clip > 0.f) {
      const float z = fminf(g[k], clip);
      g[k] = z * sigmoid_f(1.702f * z) * (fminf(fmaxf(u[k], -clip), clip) + 1.f) * r;
    } else {
      const float z = g[k] * r;
      g[k] = z * sigmoid_f(z) * (u[k] * r);
    }
  }
  Vec<T, VEC>::store(out + t * I + c, g);
}

// --------------------------------------------------------------------------------------------- query / key / value preparation
// A unit is one head row of one token: H query heads, G key heads, G value heads. L lanes share a unit; with VEC = 8 a lane
// holds eight consecutive dimensions, so rotated pairs never leave it.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
qkv_prep_kernel(const VbQkvPrep a, int L, long long units) {
  const long long u = (blockIdx.x * 256ll + threadIdx.x) / L;
  const int lane = threadIdx.x & (L - 1);
  const bool live = u < units;
  const int per = a.H + 2 * a.G;
  const long long t = live ? u / per : 0;
  const int k = live ? static_cast<int>(u % per) : 0;
  const bool is_q = k < a.H, is_v = k >= a.H + a.G;
  const int n = is_v ? a.vdim : a.dim;
  const int col = is_v ? (a.H + a.G) * a.dim + (k - a.H - a.G) * a.vdim : k * a.dim;
  const T* src = reinterpret_cast<const T*>(a.p) + t * a.ldp + col;
  const int width = a.G * (a.dim + a.vdim);
  // destinations: the query tensor, or the row in `rows` and / or the page
  T *d0 = nullptr, *d1 = nullptr;
  if (is_q) {
    d0 = reinterpret_cast<T*>(a.q) + (t * a.H + k) * a.dim;
  } else {
    const int at = is_v ? a.G * a.dim + (k - a.H - a.G) * a.vdim : (k - a.H) * a.dim;
    if (a.rows != nullptr) d0 = reinterpret_cast<T*>(a.rows) + t * a.ldr + at;
    if (a.pages != nullptr) {
      const long long sl = a.slot[t];
      if (sl >= 0 && sl < a.num_slots) d1 = reinterpret_cast<T*>(a.pages) + (sl / a.block_size) * a.page_stride + (sl % a.block_size) * width + at;
    }
  }
  float ss = 0.f, v[VEC], g[VEC], o[VEC];
  if (live && !is_v) {
    for (int c = lane * VEC; c < n; c += L * VEC) {
      Vec<T, VEC>::load(src + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += v[i] * v[i];
    }
  }
  for (int s = L >> 1; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!live) return;
  if (is_v) {
    const bool mix = a.vfirst != nullptr;
    const float lam = mix ? to_f(*reinterpret_cast<const T*>(a.vmix)) : 0.f;
    const T* first = reinterpret_cast<const T*>(a.vfirst) + t * a.ldvf + (k - a.H - a.G) * a.vdim;
    for (int c = lane * VEC; c < n; c += L * VEC) {
      Vec<T, VEC>::load(src + c, v);
      if (mix) {
        Vec<T, VEC>::load(first + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = (1.f - lam) * v[i] + lam * g[i];
      }
      if (d0 != nullptr) Vec<T, VEC>::store(d0 + c, v);
      if (d1 != nullptr) Vec<T, VEC>::store(d1 + c, v);
    }
    return;
  }
  const float r = 1.f / sqrtf(ss / n + a.eps);
  const T* nw = reinterpret_cast<const T*>(is_q ? a.qn : a.kn);
  const long long tab = static_cast<long long>(min(max(a.pos[t], 0), a.max_pos - 1)) * a.half;
  for (int c = lane * VEC; c < n; c += L * VEC) {
    Vec<T, VEC>::load(src + c, v);
    Vec<T, VEC>::load(nw + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) o[i] = v[i] * r * g[i];
    if constexpr (VEC == 1) {
      if (c < 2 * a.half) {
        const float w = to_f(src[c ^ 1]) * r * to_f(nw[c ^ 1]), cs = a.cos_t[tab + (c >> 1)], sn = a.sin_t[tab + (c >> 1)];
        o[0] = (c & 1) ? o[0] * cs + w * sn : o[0] * cs - w * sn;
      }
    } else {
#pragma unroll
      for (int i = 0; i < VEC; i += 2) {
        if (c + i < 2 * a.half) {
          const float cs = a.cos_t[tab + ((c + i) >> 1)], sn = a.sin_t[tab + ((c + i) >> 1)];
          const float x = o[i], y = o[i + 1];
          o[i] = x * cs - y * sn;
          o[i + 1] = y * cs + x * sn;
        }
      }
    }
    if (d0 != nullptr) Vec<T, VEC>::store(d0 + c, o);
    if (d1 != nullptr) Vec<T, VEC>::store(d1 + c, o);
  }
}

// --------------------------------------------------------------------------------------------- tanh of some columns, in place
template <typename T>
__global__ void __launch_bounds__(256) tanh_cols_kernel(T* __restrict__ x, long long ld, int n, long long total) {
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= total) return;
  T* at = x + i / n * ld + i % n;
  *at = from_f<T>(tanhf(to_f(*at)));
}

static bool mis16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) != 0; }

}  // namespace vb

using namespace vb;

extern "C" int vb_embed_rms(int dtype, const long long* ids, const void* w, float scale, const void* nw, float eps, float* x, void* h, int T, int W, int V,
                            cudaStream_t s) {
  if (T <= 0) return 0;
  const int thr = W >= 2048 ? 256 : 128;
  const bool vec = W % 8 == 0 && !mis16(w) && !mis16(nw);
  auto go = [&](auto kern, auto* tag) {
    typedef std::remove_pointer_t<decltype(tag)> E;
    kern<<<T, thr, 0, s>>>(ids, (const E*)w, scale, (const E*)nw, eps, x, (E*)h, W, V);
    return static_cast<int>(cudaGetLastError());
  };
  if (dtype == 0) return vec ? go(embed_rms_kernel<float, 8>, (float*)nullptr) : go(embed_rms_kernel<float, 1>, (float*)nullptr);
  return vec ? go(embed_rms_kernel<bf16, 8>, (bf16*)nullptr) : go(embed_rms_kernel<bf16, 1>, (bf16*)nullptr);
}

extern "C" int vb_residual_rms(int dtype, const VbResidRms* p, cudaStream_t s) {
  if (p->T <= 0) return 0;
  const bool vec = p->W % 8 == 0 && p->ldy % 8 == 0 && p->split_stride % 8 == 0 && p->ldr % 8 == 0 && !mis16(p->x) && !mis16(p->y) && !mis16(p->rows) &&
                   !mis16(p->nw) && !mis16(p->next) && !mis16(p->h);
  if (dtype == 0) return vec ? residual_rms<float, 8>(p, s) : residual_rms<float, 1>(p, s);
  return vec ? residual_rms<bf16, 8>(p, s) : residual_rms<bf16, 1>(p, s);
}

extern "C" int vb_gated_silu(int dtype, const void* gu, long long ldg, const float* row_scale, float clip, void* out, int T, int I, cudaStream_t s) {
  if (T <= 0 || I <= 0) return 0;
  const bool vec = I % 8 == 0 && ldg % 8 == 0 && !mis16(gu) && !mis16(out);
  const long long total = static_cast<long long>(T) * (vec ? I / 8 : I);
  const unsigned grid = static_cast<unsigned>((total + 255) / 256);
  if (dtype == 0) {
    if (vec) gated_silu_kernel<float, 8><<<grid, 256, 0, s>>>((const float*)gu, ldg, row_scale, clip, (float*)out, I, total);
    else gated_silu_kernel<float, 1><<<grid, 256, 0, s>>>((const float*)gu, ldg, row_scale, clip, (float*)out, I, total);
  } else {
    if (vec) gated_silu_kernel<bf16, 8><<<grid, 256, 0, s>>>((const bf16*)gu, ldg, row_scale, clip, (bf16*)out, I, total);
    else gated_silu_kernel<bf16, 1><<<grid, 256, 0, s>>>((const bf16*)gu, ldg, row_scale, clip, (bf16*)out, I, total);
  }
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_residual_dyt(int dtype, const VbResidDyt* p, cudaStream_t s) {
  if (p->T <= 0) return 0;
  const bool vec = p->W % 8 == 0 && p->ldr % 8 == 0 && !mis16(p->x) && !mis16(p->rows) && !mis16(p->pw) && !mis16(p->pb) && !mis16(p->nw) && !mis16(p->nb) &&
                   !mis16(p->h);
  const long long total = static_cast<long long>(p->T) * (vec ? p->W / 8 : p->W);
  const unsigned grid = static_cast<unsigned>((total + 255) / 256);
  if (dtype == 0) {
    if (vec) residual_dyt_kernel<float, 8><<<grid, 256, 0, s>>>(*p, total);
    else residual_dyt_kernel<float, 1><<<grid, 256, 0, s>>>(*p, total);
  } else {
    if (vec) residual_dyt_kernel<bf16, 8><<<grid, 256, 0, s>>>(*p, total);
    else residual_dyt_kernel<bf16, 1><<<grid, 256, 0, s>>>(*p, total);
  }
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_tanh_cols(int dtype, void* x, long long ld, int T, int n, cudaStream_t s) {
  const long long total = static_cast<long long>(T) * n;
  if (total <= 0) return 0;
  const unsigned grid = static_cast<unsigned>((total + 255) / 256);
  if (dtype == 0) tanh_cols_kernel<float><<<grid, 256, 0, s>>>((float*)x, ld, n, total);
  else tanh_cols_kernel<bf16><<<grid, 256, 0, s>>>((bf16*)x, ld, n, total);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_whole_norm(int dtype, const VbWholeNorm* p, cudaStream_t s) {
  if (p->T <= 0) return 0;
  const bool vec = p->dim % 8 == 0 && p->vdim % 8 == 0 && p->ldp % 8 == 0 && p->ldr % 8 == 0 && p->page_stride % 8 == 0 && !mis16(p->p) && !mis16(p->qn) &&
                   !mis16(p->kn) && !mis16(p->q) && !mis16(p->rows) && !mis16(p->pages);
  if (dtype == 0) {
    if (vec) whole_norm_kernel<float, 8><<<p->T, 256, 0, s>>>(*p);
    else whole_norm_kernel<float, 1><<<p->T, 256, 0, s>>>(*p);
  } else {
    if (vec) whole_norm_kernel<bf16, 8><<<p->T, 256, 0, s>>>(*p);
    else whole_norm_kernel<bf16, 1><<<p->T, 256, 0, s>>>(*p);
  }
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_diff_combine(int dtype, const void* a, int a_f32, const void* vec, int dim, float diff, float eps, void* out, int T, int H, int dv, cudaStream_t s) {
  const long long rows = static_cast<long long>(T) * H;
  if (rows <= 0) return 0;
  const unsigned grid = static_cast<unsigned>((rows + 3) / 4);
  if (dtype == 0) diff_combine_kernel<float, float><<<grid, 128, 0, s>>>((const float*)a, (const float*)vec, dim, diff, eps, (float*)out, rows, dv);
  else if (a_f32) diff_combine_kernel<float, bf16><<<grid, 128, 0, s>>>((const float*)a, (const bf16*)vec, dim, diff, eps, (bf16*)out, rows, dv);
  else diff_combine_kernel<bf16, bf16><<<grid, 128, 0, s>>>((const bf16*)a, (const bf16*)vec, dim, diff, eps, (bf16*)out, rows, dv);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_gated_rms(int dtype, const void* o, long long ldo, const void* g, long long ldg, const void* norm, float eps, void* out, int T, int W, int heads,
                            cudaStream_t s) {
  if (T <= 0 || W <= 0) return 0;
  if (heads > 1) {
    const int n = W / heads;
    const bool v8 = n % 8 == 0 && ldo % 8 == 0 && ldg % 8 == 0 && !mis16(o) && !mis16(g) && !mis16(norm) && !mis16(out);
    if (dtype == 0) return v8 ? gated_rms_heads<float, 8>(o, ldo, g, ldg, norm, eps, out, T, n, heads, s) : gated_rms_heads<float, 1>(o, ldo, g, ldg, norm, eps, out, T, n, heads, s);
    return v8 ? gated_rms_heads<bf16, 8>(o, ldo, g, ldg, norm, eps, out, T, n, heads, s) : gated_rms_heads<bf16, 1>(o, ldo, g, ldg, norm, eps, out, T, n, heads, s);
  }
  const bool vec = W % 8 == 0 && ldo % 8 == 0 && ldg % 8 == 0 && !mis16(o) && !mis16(g) && !mis16(norm) && !mis16(out);
  if (dtype == 0) return vec ? gated_rms<float, 8>(o, ldo, g, ldg, norm, eps, out, T, W, s) : gated_rms<float, 1>(o, ldo, g, ldg, norm, eps, out, T, W, s);
  return vec ? gated_rms<bf16, 8>(o, ldo, g, ldg, norm, eps, out, T, W, s) : gated_rms<bf16, 1>(o, ldo, g, ldg, norm, eps, out, T, W, s);
}

extern "C" int vb_qkv_prep(int dtype, const VbQkvPrep* p, cudaStream_t s) {
  if (p->T <= 0) return 0;
  const bool vec = p->dim % 8 == 0 && p->vdim % 8 == 0 && p->ldp % 8 == 0 && p->ldvf % 8 == 0 && p->ldr % 8 == 0 && p->page_stride % 8 == 0 && !mis16(p->p) &&
                   !mis16(p->qn) && !mis16(p->kn) && !mis16(p->vfirst) && !mis16(p->q) && !mis16(p->rows) && !mis16(p->pages);
  const int most = p->dim > p->vdim ? p->dim : p->vdim;
  int L = 1;
  while (L < 32 && L * (vec ? 8 : 1) < most) L *= 2;
  const long long units = static_cast<long long>(p->T) * (p->H + 2 * p->G);
  const unsigned grid = static_cast<unsigned>((units * L + 255) / 256);
  if (dtype == 0) {
    if (vec) qkv_prep_kernel<float, 8><<<grid, 256, 0, s>>>(*p, L, units);
    else qkv_prep_kernel<float, 1><<<grid, 256, 0, s>>>(*p, L, units);
  } else {
    if (vec) qkv_prep_kernel<bf16, 8><<<grid, 256, 0, s>>>(*p, L, units);
    else qkv_prep_kernel<bf16, 1><<<grid, 256, 0, s>>>(*p, L, units);
  }
  return static_cast<int>(cudaGetLastError());
}
