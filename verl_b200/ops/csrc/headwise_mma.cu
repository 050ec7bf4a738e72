// Per-head products of the decode step: out[m, h, :] = a[m, h, :] w[h]^T, or a[m, h, :] w[h] for weights stored [H, K, N]
// (the absorbed key expansion), optionally times sigmoid(gate[m, h]); the absorbing form also rotates the query's positional
// part and puts it behind the product. The heads' weights are read once and dominate the traffic, the products are small:
// 64 tokens x 64 columns per CTA on m16n8k16 MMAs, K in steps of 64 through a two-stage cp.async ring.
// Compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

namespace vb {

typedef __nv_bfloat16 bf16;
constexpr int HW_T = 64, HW_P = 72;  // tile edge, row pitch (elements) that keeps ldmatrix free of bank conflicts

__device__ __forceinline__ uint32_t hw_smem(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void hw_cp16(void* dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(hw_smem(dst)), "l"(src), "r"(ok ? 16 : 0));
}
__device__ __forceinline__ void hw_ldsm(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void hw_ldsm_t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void hw_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <bool KN>
__global__ void __launch_bounds__(128)
headwise_kernel(const VbHeadwise p) {
  __shared__ __align__(16) bf16 sA[2][HW_T * HW_P], sB[2][HW_T * HW_P];
  const int h = blockIdx.z, m0 = blockIdx.y * HW_T, n0 = blockIdx.x * HW_T, tid = threadIdx.x;
  const bf16* A = reinterpret_cast<const bf16*>(p.a) + static_cast<long long>(h) * p.a_head;
  const bf16* B = reinterpret_cast<const bf16*>(p.w) + static_cast<long long>(h) * p.w_head;
  bf16* O = reinterpret_cast<bf16*>(p.out) + static_cast<long long>(h) * p.o_head;
  if (n0 >= p.N) {  // the positional part: pairs (2i, 2i + 1) of the first 2 * half dimensions turn, the rest is copied
    const int hp = (p.rot + 1) / 2, per = hp < 128 ? 128 / hp : 1;   // pairs per row, rows per round
    for (int c2 = tid % hp; c2 < hp && tid / hp < per; c2 += 128) {
#pragma unroll 4
      for (int r = tid / hp; r < HW_T; r += per) {
        const int m = m0 + r, c = 2 * c2;
        if (m >= p.M) continue;
        const bf16* src = A + m * p.lda + p.K + c;
        bf16* dst = O + m * p.ldo + p.N + c;
        const float u = to_f(src[0]), v = c + 1 < p.rot ? to_f(src[1]) : 0.f;
        float cc = 1.f, ss = 0.f;
        if (c2 < p.half) {
          const long long at = static_cast<long long>(min(max(p.pos[m], 0), p.max_pos - 1)) * p.half + c2;
          cc = p.cos_t[at];
          ss = p.sin_t[at];
        }
        dst[0] = from_f<bf16>(u * cc - v * ss);
        if (c + 1 < p.rot) dst[1] = from_f<bf16>(v * cc + u * ss);
      }
    }
    return;
  }
  auto load = [&](int st, int k0) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int i = tid + u * 128, r = i >> 3, c = (i & 7) * 8;
      const bool okA = m0 + r < p.M && k0 + c < p.K;
      hw_cp16(&sA[st][r * HW_P + c], okA ? A + (m0 + r) * p.lda + k0 + c : A, okA);
      if (KN) {
        const bool ok = k0 + r < p.K && n0 + c < p.N;
        hw_cp16(&sB[st][r * HW_P + c], ok ? B + (k0 + r) * p.ldw + n0 + c : B, ok);
      } else {
        const bool ok = n0 + r < p.N && k0 + c < p.K;
        hw_cp16(&sB[st][r * HW_P + c], ok ? B + (n0 + r) * p.ldw + k0 + c : B, ok);
      }
    }
    asm volatile("cp.async.commit_group;");
  };
  const int warp = tid >> 5, lane = tid & 31, wm = (warp >> 1) * 32, wn = (warp & 1) * 32, mi = lane >> 3, r8 = lane & 7;
  float acc[2][4][4] = {};
  const int steps = (p.K + HW_T - 1) / HW_T;
  load(0, 0);
  for (int k = 0; k < steps; ++k) {
    if (k + 1 < steps) {
      load((k + 1) & 1, (k + 1) * HW_T);
      asm volatile("cp.async.wait_group 1;");
    } else {
      asm volatile("cp.async.wait_group 0;");
    }
    __syncthreads();
    const uint32_t a = hw_smem(sA[k & 1]), b = hw_smem(sB[k & 1]);
#pragma unroll
    for (int kk = 0; kk < HW_T; kk += 16) {
      uint32_t fa[2][4], fb[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) hw_ldsm(fa[i], a + ((wm + i * 16 + (mi & 1) * 8 + r8) * HW_P + kk + (mi >> 1) * 8) * 2);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        // fb[j]: two 8-column blocks, each as its two k halves: {n0 k0, n0 k8, n8 k0, n8 k8}
        if (KN) hw_ldsm_t(fb[j], b + ((kk + (mi & 1) * 8 + r8) * HW_P + wn + j * 16 + (mi >> 1) * 8) * 2);
        else hw_ldsm(fb[j], b + ((wn + j * 16 + (mi >> 1) * 8 + r8) * HW_P + kk + (mi & 1) * 8) * 2);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) hw_mma(acc[i][j], fa[i], fb[j >> 1][(j & 1) * 2], fb[j >> 1][(j & 1) * 2 + 1]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int m = m0 + wm + i * 16 + half * 8 + (lane >> 2);
      if (m >= p.M) continue;
      const float g = p.gate != nullptr ? sigmoid_f(p.gate[m * p.ldg + h]) : 1.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + wn + j * 8 + (lane & 3) * 2;
        if (n >= p.N) continue;
        const __nv_bfloat162 v = __floats2bfloat162_rn(acc[i][j][2 * half] * g, acc[i][j][2 * half + 1] * g);
        *reinterpret_cast<__nv_bfloat162*>(O + m * p.ldo + n) = v;
      }
    }
}

}  // namespace vb

using namespace vb;

// Returns -1 for sizes and alignments it does not serve.
extern "C" int vb_headwise(const VbHeadwise* p, cudaStream_t s) {
  if (p->M <= 0 || p->H <= 0) return 0;
  if ((p->K | p->N | p->lda | p->a_head | p->w_head | p->ldw) % 8 || (p->ldo | p->o_head) % 2) return -1;
  if ((reinterpret_cast<uintptr_t>(p->a) | reinterpret_cast<uintptr_t>(p->w)) & 15 || (reinterpret_cast<uintptr_t>(p->out) & 3)) return -1;
  const dim3 grid((p->N + HW_T - 1) / HW_T + (p->rot > 0 ? 1 : 0), (p->M + HW_T - 1) / HW_T, p->H);
  if (grid.y > 65535 || grid.z > 65535) return -1;
  if (p->kn) headwise_kernel<true><<<grid, 128, 0, s>>>(*p);
  else headwise_kernel<false><<<grid, 128, 0, s>>>(*p);
  return static_cast<int>(cudaGetLastError());
}
