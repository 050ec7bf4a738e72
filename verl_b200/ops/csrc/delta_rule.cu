// Generalized delta rule, S = diag(w) S - (a u)(u^T S) + k v^T, o = S^T r per head: single step for decoding (with the head's output norm
// and gate), and token-by-token scan of prompts (32-bit mode, and sizes the chunked kernel does not serve). The state [d, d] is read and
// written once per step; the removal reads it before it is updated, so a thread holds its part of the state in registers.
// Decays, rates, unit keys and the state are fp32; compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>

namespace vb {

typedef __nv_bfloat16 bf16;

constexpr float DR_FALL = 0.60653065971263342f;   // exp(-1/2): a decay never falls below exp(-exp(-1/2))

__device__ __forceinline__ float dr_decay(float z) { return expf(-DR_FALL * sigmoid_f(z)); }

// One CTA = (slot, head). Threads form RG row groups x (d / VEC) column groups; a thread owns VEC columns of its ROWS rows
// (row = i * RG + group), which stay in registers between the two passes over them.
template <typename T, int VEC, int ROWS>
__global__ void __launch_bounds__(256)
delta_decode_kernel(const VbDelta p, int RG) {
  extern __shared__ float sm[];
  __shared__ float red[33];
  const int h = blockIdx.x, tid = threadIdx.x, d = p.d, W = p.H * d;
  const long long t = blockIdx.y;
  const int col0 = h * d;
  T* orow = reinterpret_cast<T*>(p.out) + t * p.ldo + col0;
  if (!p.active[t]) {
    for (int c = tid; c < d; c += blockDim.x) orow[c] = from_f<T>(0.f);
    return;
  }
  float *sr = sm, *sk = sr + d, *sw = sk + d, *sb = sw + d, *part = sb + d, *part2 = part + RG * d;   // [d] each, then [RG][d] twice
  const int cg = d / VEC, rg = tid / cg, ct = tid % cg, lane = tid & 31;
  const bool on = rg < RG;
  float* S = p.state + t * p.slot_stride + static_cast<long long>(h) * d * d + ct * VEC;
  const T* row = reinterpret_cast<const T*>(p.p) + t * p.ldp + col0;
  const T* zw = reinterpret_cast<const T*>(p.zw) + t * p.ldz + col0;
  float s[ROWS][VEC], v[VEC] = {}, gate[VEC] = {}, nrm[VEC] = {};
  if (on) {
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
      if (i * RG + rg < d) Vec<float, VEC>::load(S + static_cast<long long>(i * RG + rg) * d, s[i]);
    Vec<T, VEC>::load(row + 2 * W + ct * VEC, v);
    if (rg == 0) {
      Vec<T, VEC>::load(row + 4 * W + ct * VEC, gate);
      Vec<T, VEC>::load(reinterpret_cast<const T*>(p.norm) + col0 + ct * VEC, nrm);
    }
  }
  float kk = 0.f;                                    // every warp sums up the whole key
  for (int c = lane; c < d; c += 32) {
    const float k = to_f(row[W + c]);
    kk += k * k;
  }
  for (int c = tid; c < d; c += blockDim.x) {
    const float k = to_f(row[W + c]);
    sr[c] = to_f(row[c]);
    sk[c] = k;
    sw[c] = dr_decay(to_f(zw[c]) + to_f(reinterpret_cast<const T*>(p.w0)[col0 + c]));
    sb[c] = sigmoid_f(to_f(row[3 * W + c]) + to_f(reinterpret_cast<const T*>(p.ab)[col0 + c])) * k;
  }
  const float iu2 = 1.f / (warp_sum(kk) + 1e-6f);    // both factors of the removal carry the key's length
  __syncthreads();
  float held[VEC] = {}, o[VEC] = {};
  if (on) {
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int r = i * RG + rg;
      if (r < d) {
        const float k_ = sk[r];
#pragma unroll
        for (int k = 0; k < VEC; ++k) held[k] = fmaf(k_, s[i][k], held[k]);
      }
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) part[rg * d + ct * VEC + k] = held[k];
  }
  __syncthreads();
  if (on) {
#pragma unroll
    for (int k = 0; k < VEC; ++k) held[k] = 0.f;
    for (int g = 0; g < RG; ++g)
#pragma unroll
      for (int k = 0; k < VEC; ++k) held[k] += part[g * d + ct * VEC + k];
#pragma unroll
    for (int k = 0; k < VEC; ++k) held[k] *= iu2;
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int r = i * RG + rg;
      if (r < d) {
        const float w = sw[r], b = sb[r], kx = sk[r], q = sr[r];
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
          s[i][k] = fmaf(w, s[i][k], fmaf(kx, v[k], -b * held[k]));
          o[k] = fmaf(q, s[i][k], o[k]);
        }
        Vec<float, VEC>::store(S + static_cast<long long>(r) * d, s[i]);
      }
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) part2[rg * d + ct * VEC + k] = o[k];
  }
  __syncthreads();
  float ss = 0.f;
  if (on && rg == 0) {
#pragma unroll
    for (int k = 0; k < VEC; ++k) o[k] = 0.f;
    for (int g = 0; g < RG; ++g)
#pragma unroll
      for (int k = 0; k < VEC; ++k) o[k] += part2[g * d + ct * VEC + k];
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss += o[k] * o[k];
  }
  if (cg <= 32) {                                    // the columns' threads are one warp
    if (tid >= 32) return;
    ss = warp_sum(ss);
  } else {
    ss = block_sum(ss, red);
  }
  const float r = 1.f / sqrtf(ss / d + p.eps);
  if (on && rg == 0) {
#pragma unroll
    for (int k = 0; k < VEC; ++k) orow[ct * VEC + k] = from_f<T>(o[k] * r * nrm[k] * sigmoid_f(gate[k]));
  }
}

// Heads too large for registers: a thread owns every 256th column and reads its part of the state twice.
template <typename T>
__global__ void __launch_bounds__(256)
delta_decode_any_kernel(const VbDelta p) {
  extern __shared__ float sm[];
  __shared__ float red[33];
  const int h = blockIdx.x, tid = threadIdx.x, d = p.d, W = p.H * d, col0 = h * d;
  const long long t = blockIdx.y;
  T* orow = reinterpret_cast<T*>(p.out) + t * p.ldo + col0;
  if (!p.active[t]) {
    for (int c = tid; c < d; c += 256) orow[c] = from_f<T>(0.f);
    return;
  }
  float *sr = sm, *sk = sr + d, *sw = sk + d, *sb = sw + d, *so = sb + d;   // [d] each
  float* S = p.state + t * p.slot_stride + static_cast<long long>(h) * d * d;
  const T* row = reinterpret_cast<const T*>(p.p) + t * p.ldp + col0;
  const T* zw = reinterpret_cast<const T*>(p.zw) + t * p.ldz + col0;
  float kk = 0.f;
  for (int c = tid; c < d; c += 256) {
    const float k = to_f(row[W + c]);
    sr[c] = to_f(row[c]);
    sk[c] = k;
    sw[c] = dr_decay(to_f(zw[c]) + to_f(reinterpret_cast<const T*>(p.w0)[col0 + c]));
    sb[c] = sigmoid_f(to_f(row[3 * W + c]) + to_f(reinterpret_cast<const T*>(p.ab)[col0 + c])) * k;
    kk += k * k;
  }
  const float iu2 = 1.f / (block_sum(kk, red) + 1e-6f);
  float ss = 0.f;
  for (int c = tid; c < d; c += 256) {
    float held = 0.f, o = 0.f;
    const float v = to_f(row[2 * W + c]);
    for (int r = 0; r < d; ++r) held = fmaf(sk[r], S[static_cast<long long>(r) * d + c], held);
    held *= iu2;
    for (int r = 0; r < d; ++r) {
      float* at = S + static_cast<long long>(r) * d + c;
      const float s = fmaf(sw[r], *at, fmaf(sk[r], v, -sb[r] * held));
      *at = s;
      o = fmaf(sr[r], s, o);
    }
    so[c] = o;
    ss += o * o;
  }
  const float f = 1.f / sqrtf(block_sum(ss, red) / d + p.eps);
  for (int c = tid; c < d; c += 256) orow[c] = from_f<T>(so[c] * f * to_f(reinterpret_cast<const T*>(p.norm)[col0 + c]) * sigmoid_f(to_f(row[4 * W + c])));
}

// Token-by-token scan of a portion: one CTA = one (sequence, head, 32 columns of v); the state columns live in shared memory.
constexpr int DS_COLS = 32, DS_ROWS = 8;
template <typename T>
__global__ void __launch_bounds__(DS_COLS * DS_ROWS)
delta_scan_kernel(const VbDelta p) {
  extern __shared__ float sm[];
  __shared__ float part[DS_ROWS][DS_COLS], red[33];
  const int d = p.d, W = p.H * d;
  float *S = sm, *sr = S + d * DS_COLS, *sk = sr + d, *su = sk + d, *sw = su + d, *sb = sw + d;
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * DS_COLS, tid = threadIdx.x, c = tid % DS_COLS, rg = tid / DS_COLS, col0 = h * d;
  const bool c_ok = c0 + c < d, have = p.slots != nullptr && p.slots[b] >= 0;
  float* st = have ? p.state + static_cast<long long>(p.slots[b]) * p.slot_stride + static_cast<long long>(h) * d * d : nullptr;
  const bool zero = !have || (p.fresh != nullptr && p.fresh[b] != 0);
  for (int r = rg; r < d; r += DS_ROWS) S[r * DS_COLS + c] = (zero || !c_ok) ? 0.f : st[static_cast<long long>(r) * d + c0 + c];
  T* out = reinterpret_cast<T*>(p.out);
  auto column_sum = [&](float v) {
    part[rg][c] = v;
    __syncthreads();
    float a = 0.f;
#pragma unroll
    for (int u = 0; u < DS_ROWS; ++u) a += part[u][c];
    __syncthreads();
    return a;
  };
  for (long long t = p.cu[b]; t < p.cu[b + 1]; ++t) {
    const T* row = reinterpret_cast<const T*>(p.p) + t * p.ldp + col0;
    const T* zw = reinterpret_cast<const T*>(p.zw) + t * p.ldz + col0;
    float kk = 0.f;
    for (int r = tid; r < d; r += DS_COLS * DS_ROWS) {
      sr[r] = to_f(row[r]);
      sk[r] = to_f(row[W + r]);
      sw[r] = dr_decay(to_f(zw[r]) + to_f(reinterpret_cast<const T*>(p.w0)[col0 + r]));
      kk += sk[r] * sk[r];
    }
    const float iu = 1.f / sqrtf(block_sum(kk, red) + 1e-6f);
    for (int r = tid; r < d; r += DS_COLS * DS_ROWS) {
      const float u = sk[r] * iu;
      su[r] = u;
      sb[r] = sigmoid_f(to_f(row[3 * W + r]) + to_f(reinterpret_cast<const T*>(p.ab)[col0 + r])) * u;
    }
    __syncthreads();
    const float v = c_ok ? to_f(row[2 * W + c0 + c]) : 0.f;
    float acc = 0.f;
    for (int r = rg; r < d; r += DS_ROWS) acc = fmaf(su[r], S[r * DS_COLS + c], acc);
    const float held = column_sum(acc);
    acc = 0.f;
    for (int r = rg; r < d; r += DS_ROWS) {
      const float s = fmaf(sw[r], S[r * DS_COLS + c], fmaf(sk[r], v, -sb[r] * held));
      S[r * DS_COLS + c] = s;
      acc = fmaf(sr[r], s, acc);
    }
    const float o = column_sum(acc);                 // its second barrier also frees the vectors for the next token
    if (rg == 0 && c_ok) out[t * p.ldo + col0 + c0 + c] = from_f<T>(o);
  }
  if (have && c_ok)
    for (int r = rg; r < d; r += DS_ROWS) st[static_cast<long long>(r) * d + c0 + c] = S[r * DS_COLS + c];
}

template <typename K>
static int dr_smem(K kern, int bytes) {
  if (bytes > 232448 - 4096) return -2;
  return bytes > 40 * 1024 ? static_cast<int>(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes)) : 0;
}

template <typename T, int VEC>
static int delta_decode(const VbDelta* p, cudaStream_t s) {
  const int cg = p->d / VEC;
  int RG = (p->d + 15) / 16;                         // sixteen rows of a thread: small CTAs, many of them
  if (RG * cg < 64) RG = 64 / cg;
  if (RG * cg > 256) RG = 256 / cg;
  if (RG > p->d) RG = p->d;
  const int rows = RG > 0 ? (p->d + RG - 1) / RG : p->d;
  if (RG < 1 || rows > 64) {
    const int smem = 5 * p->d * 4, rc = dr_smem(delta_decode_any_kernel<T>, smem);
    if (rc != 0) return rc;
    delta_decode_any_kernel<T><<<dim3(p->H, p->T), 256, smem, s>>>(*p);
    return static_cast<int>(cudaGetLastError());
  }
  const int smem = (4 * p->d + 2 * RG * p->d) * 4;
  auto go = [&](auto kern) {
    const int rc = dr_smem(kern, smem);
    if (rc != 0) return rc;
    kern<<<dim3(p->H, p->T), (RG * cg + 31) / 32 * 32, smem, s>>>(*p, RG);
    return static_cast<int>(cudaGetLastError());
  };
  if (rows <= 4) return go(delta_decode_kernel<T, VEC, 4>);
  if (rows <= 8) return go(delta_decode_kernel<T, VEC, 8>);
  if (rows <= 16) return go(delta_decode_kernel<T, VEC, 16>);
  return go(delta_decode_kernel<T, VEC, 64>);
}

template <typename T>
static int delta_scan(const VbDelta* p, cudaStream_t s) {
  const int smem = (p->d * DS_COLS + 5 * p->d) * 4;
  const int rc = dr_smem(delta_scan_kernel<T>, smem);
  if (rc != 0) return rc;
  delta_scan_kernel<T><<<dim3((p->d + DS_COLS - 1) / DS_COLS, p->H, p->B), DS_COLS * DS_ROWS, smem, s>>>(*p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace vb

using namespace vb;

extern "C" int vb_delta_decode(int dtype, const VbDelta* p, cudaStream_t s) {
  if (p->T <= 0) return 0;
  if (p->T > 65535) return -1;
  const bool v4 = p->d % 4 == 0 && p->slot_stride % 4 == 0 && !(reinterpret_cast<uintptr_t>(p->state) & 15) &&
                  (dtype == 1 || (p->ldp % 4 == 0 && !(reinterpret_cast<uintptr_t>(p->p) & 15) && !(reinterpret_cast<uintptr_t>(p->norm) & 15)));
  if (dtype == 0) return v4 ? delta_decode<float, 4>(p, s) : delta_decode<float, 1>(p, s);
  return v4 ? delta_decode<bf16, 4>(p, s) : delta_decode<bf16, 1>(p, s);
}

extern "C" int vb_delta_scan(int dtype, const VbDelta* p, cudaStream_t s) {
  if (p->T <= 0 || p->B <= 0) return 0;
  if (p->B > 65535 || p->H > 65535) return -1;
  return dtype == 0 ? delta_scan<float>(p, s) : delta_scan<bf16>(p, s);
}
