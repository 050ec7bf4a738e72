// Linear recurrence with one fixed decay per head (S = decay S + k v^T, o = S^T q): single step for decoding and token-by-token scan
// (32-bit mode, and sizes the chunked kernel does not serve). State in fp32; compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>

namespace vb {

typedef __nv_bfloat16 bf16;

// One CTA = (slot, head): the state is read and written once. A thread owns VEC columns of v and every rgs-th row.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
lightning_decode_kernel(const VbLightning p) {
  extern __shared__ float sm[];
  const int h = blockIdx.x, tid = threadIdx.x, d = p.d, e = p.e, H = p.H;
  const long long t = blockIdx.y;
  T* orow = reinterpret_cast<T*>(p.out) + t * p.ldo + static_cast<long long>(h) * e;
  if (!p.active[t]) {
    for (int c = tid; c < e; c += blockDim.x) orow[c] = from_f<T>(0.f);
    return;
  }
  float *sq = sm, *sk = sq + d, *so = sk + d;         // [d], [d], [row groups][e]
  float* S = p.state + t * p.slot_stride + static_cast<long long>(h) * d * e;
  const T* row = reinterpret_cast<const T*>(p.p) + t * p.ldp;
  const float keep = p.decay[h];
  const int cg = (e + VEC - 1) / VEC, tpc = min(cg, static_cast<int>(blockDim.x)), rgs = blockDim.x / tpc, rg = tid / tpc, ct = tid % tpc;
  const T* vrow = row + 2 * H * d + static_cast<long long>(h) * e;
  constexpr int U = 8;                                // rows in flight
  for (int r = tid; r < d; r += blockDim.x) {
    sq[r] = to_f(row[h * d + r]);
    sk[r] = to_f(row[(H + h) * d + r]);
  }
  __syncthreads();
  if (rg < rgs) {
    for (int c = ct; c < cg; c += tpc) {
      float v[VEC], o[VEC] = {};
      Vec<T, VEC>::load(vrow + c * VEC, v);
      float* Sc = S + c * VEC;
      for (int r0 = rg; r0 < d; r0 += U * rgs) {
        float s[U][VEC];
#pragma unroll
        for (int u = 0; u < U; ++u)
          if (r0 + u * rgs < d) Vec<float, VEC>::load(Sc + static_cast<long long>(r0 + u * rgs) * e, s[u]);
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = r0 + u * rgs;
          if (r >= d) break;
          const float k = sk[r], q = sq[r];
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            s[u][i] = keep * s[u][i] + k * v[i];
            o[i] += s[u][i] * q;
          }
          Vec<float, VEC>::store(Sc + static_cast<long long>(r) * e, s[u]);
        }
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) so[rg * e + c * VEC + i] = o[i];
    }
  }
  __syncthreads();
  for (int c = tid; c < e; c += blockDim.x) {
    float o = 0.f;
    for (int u = 0; u < rgs; ++u) o += so[u * e + c];
    orow[c] = from_f<T>(o);
  }
}

// Token-by-token scan of a portion: one CTA = one (sequence, head, 32 columns of v); the state columns live in shared memory.
constexpr int LS_COLS = 32, LS_ROWS = 8;
template <typename T>
__global__ void __launch_bounds__(LS_COLS * LS_ROWS)
lightning_scan_kernel(const VbLightning p) {
  extern __shared__ float sm[];
  __shared__ float part[LS_ROWS][LS_COLS];
  const int d = p.d, e = p.e, H = p.H;
  float *S = sm, *sq = S + d * LS_COLS, *sk = sq + d;  // [d][32], [d], [d]
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * LS_COLS, c = threadIdx.x, rg = threadIdx.y, tid = rg * LS_COLS + c;
  const bool c_ok = c0 + c < e, have = p.slots != nullptr && p.slots[b] >= 0;
  float* st = have ? p.state + static_cast<long long>(p.slots[b]) * p.slot_stride + static_cast<long long>(h) * d * e : nullptr;
  const bool zero = !have || (p.fresh != nullptr && p.fresh[b] != 0);
  for (int r = rg; r < d; r += LS_ROWS) S[r * LS_COLS + c] = (zero || !c_ok) ? 0.f : st[static_cast<long long>(r) * e + c0 + c];
  const float keep = p.decay[h];
  T* out = reinterpret_cast<T*>(p.out);
  for (long long t = p.cu[b]; t < p.cu[b + 1]; ++t) {
    const T* row = reinterpret_cast<const T*>(p.p) + t * p.ldp;
    for (int r = tid; r < d; r += LS_COLS * LS_ROWS) {
      sq[r] = to_f(row[h * d + r]);
      sk[r] = to_f(row[(H + h) * d + r]);
    }
    __syncthreads();
    const float v = c_ok ? to_f(row[2 * H * d + h * e + c0 + c]) : 0.f;
    float acc = 0.f;
    for (int r = rg; r < d; r += LS_ROWS) {
      const float s = keep * S[r * LS_COLS + c] + sk[r] * v;
      S[r * LS_COLS + c] = s;
      acc += s * sq[r];
    }
    part[rg][c] = acc;
    __syncthreads();
    if (rg == 0 && c_ok) {
      float o = 0.f;
#pragma unroll
      for (int u = 0; u < LS_ROWS; ++u) o += part[u][c];
      out[t * p.ldo + static_cast<long long>(h) * e + c0 + c] = from_f<T>(o);
    }
    // the next token's q and k are written behind this barrier's pair: `part` and the rows have been read by then
    __syncthreads();
  }
  if (have && c_ok)
    for (int r = rg; r < d; r += LS_ROWS) st[static_cast<long long>(r) * e + c0 + c] = S[r * LS_COLS + c];
}

template <typename K>
static int ln_smem(K kern, int bytes) {
  if (bytes > 232448 - 4096) return -2;
  return bytes > 40 * 1024 ? static_cast<int>(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes)) : 0;
}

template <typename T, int VEC>
static int lightning_decode(const VbLightning* p, cudaStream_t s) {
  const int cg = (p->e + VEC - 1) / VEC, tpc = cg < 256 ? cg : 256, rgs = 256 / tpc, smem = (2 * p->d + rgs * p->e) * 4;
  const int rc = ln_smem(lightning_decode_kernel<T, VEC>, smem);
  if (rc != 0) return rc;
  lightning_decode_kernel<T, VEC><<<dim3(p->H, p->T), 256, smem, s>>>(*p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int lightning_scan(const VbLightning* p, cudaStream_t s) {
  const int smem = (p->d * LS_COLS + 2 * p->d) * 4;
  const int rc = ln_smem(lightning_scan_kernel<T>, smem);
  if (rc != 0) return rc;
  lightning_scan_kernel<T><<<dim3((p->e + LS_COLS - 1) / LS_COLS, p->H, p->B), dim3(LS_COLS, LS_ROWS), smem, s>>>(*p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace vb

using namespace vb;

extern "C" int vb_lightning_decode(int dtype, const VbLightning* p, cudaStream_t s) {
  if (p->T <= 0) return 0;
  if (p->T > 65535) return -1;
  const bool v4 = p->e % 4 == 0 && p->slot_stride % 4 == 0 && !(reinterpret_cast<uintptr_t>(p->state) & 15);
  if (dtype == 0) {
    const bool p4 = p->ldp % 4 == 0 && (2 * p->H * p->d) % 4 == 0 && !(reinterpret_cast<uintptr_t>(p->p) & 15);
    return v4 && p4 ? lightning_decode<float, 4>(p, s) : lightning_decode<float, 1>(p, s);
  }
  return v4 ? lightning_decode<bf16, 4>(p, s) : lightning_decode<bf16, 1>(p, s);
}

extern "C" int vb_lightning_scan(int dtype, const VbLightning* p, cudaStream_t s) {
  if (p->T <= 0 || p->B <= 0) return 0;
  if (p->B > 65535 || p->H > 65535) return -1;
  return dtype == 0 ? lightning_scan<float>(p, s) : lightning_scan<bf16>(p, s);
}
