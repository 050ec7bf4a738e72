// Lightning recurrence over prompts for query / key sizes of 129 to 256 (lightning_tcgen05.cu serves the others), 64 tokens at a time on
// m16n8k16 MMAs (bf16 q, k, v; fp32 state).
//
// With the head's fixed decay l, inside a chunk
//   o_t = l^(t + 1) q_t S_prev + sum_{s <= t} l^(t - s) (q_t . k_s) v_s
//   S_C = l^C S_prev + sum_s l^(C - 1 - s) k_s v_s^T
// so a chunk is four small products. One CTA = (sequence segment, head, up to 128 columns of v); a warp owns 16 columns and keeps
// their part of S^T in fp32 accumulators for the whole segment. The accumulator layout of S^T is the B-operand layout of the read-out, so
// S never leaves the registers; fp32 values that enter an MMA (S, the weighted scores, v weighted by the decay) are split into two
// bf16 terms, which keeps 16 mantissa bits. Chunks come through two shared-memory stages (cp.async, 16-byte pieces swizzled
// by row); two barriers per chunk.
//
// Sequences are cut into segments when there are too few of them for the GPU: a first launch (FULL = false) computes every segment's
// own contribution to the state from nothing, the second starts each segment from the fold of those before it. Compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>

namespace vb {

typedef __nv_bfloat16 bf16;
constexpr int LC_C = 64;   // tokens per chunk

__device__ __forceinline__ uint32_t lc_smem(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void lc_cp16(uint32_t dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0));
}
__device__ __forceinline__ void lc_ldsm(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void lc_ldsm_t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void lc_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two floats as bf16 pair plus the pair of what rounding dropped
__device__ __forceinline__ void lc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
// byte offset of 16-byte piece `c` of row `r`; rows of ROW bytes (a multiple of 128)
template <int ROW>
__device__ __forceinline__ uint32_t lc_at(int r, int c) { return static_cast<uint32_t>(r * ROW + ((c ^ (r & 7)) << 4)); }

template <int DP, int EW>
struct LcSmem {
  static constexpr int QB = LC_C * DP * 2, VB = LC_C * EW * 32;     // bytes of a chunk of q (or k), of v
  static constexpr int STAGE = 2 * QB + VB;
  static constexpr int OFF_P = 2 * STAGE;                           // weighted scores in two bf16 terms
  static constexpr int OFF_D = OFF_P + 2 * LC_C * LC_C * 2;         // powers of the decay, 0 .. 64
  static constexpr int TOTAL = OFF_D + 80 * 4;
};

template <int DP, int EW, bool FULL>
__global__ void __launch_bounds__(32 * EW, 1)
lightning_chunk_kernel(const VbLightning P, int nseg, float* __restrict__ local) {
  using L = LcSmem<DP, EW>;
  constexpr int THREADS = 32 * EW, NT = DP / 8, KS = DP / 16, QROW = DP * 2, VROW = EW * 32, PROW = LC_C * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  float* dec = reinterpret_cast<float*>(smem + L::OFF_D);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, er = lane >> 2, kc = (lane & 3) * 2, mi = lane >> 3, r8 = lane & 7;
  const int b = blockIdx.z / nseg, seg = blockIdx.z % nseg, h = blockIdx.y, c0 = blockIdx.x * (EW * 16);
  const int H = P.H, d = P.d, e = P.e;
  const int s0 = P.cu[b], len = P.cu[b + 1] - s0;
  const int seg_len = ((len + nseg - 1) / nseg + LC_C - 1) / LC_C * LC_C;
  const int t_lo = seg * seg_len, t_hi = min(len, t_lo + seg_len);
  if (t_lo >= t_hi) return;
  if (!FULL && t_hi == len) return;                  // nothing follows: the segment's own state is not needed
  const int e0 = c0 + warp * 16;
  const bool have = P.slots != nullptr && P.slots[b] >= 0;
  float* slot = have ? P.state + static_cast<long long>(P.slots[b]) * P.slot_stride + static_cast<long long>(h) * d * e : nullptr;
  const float lam = P.decay[h];
  for (int i = tid; i <= LC_C; i += THREADS) dec[i] = i == 0 ? 1.f : powf(lam, static_cast<float>(i));

  const bf16* base = reinterpret_cast<const bf16*>(P.p) + static_cast<long long>(s0) * P.ldp;
  const int vw = min(EW * 16, e - c0) / 8;           // 16-byte pieces of a v row
  auto load = [&](int st, int t0) {
    const uint32_t q = lc_smem(smem + st * L::STAGE), k = q + L::QB, v = k + L::QB;
    for (int i = tid; i < LC_C * (DP / 8); i += THREADS) {
      const int r = i / (DP / 8), c = i % (DP / 8);
      const bool ok = t0 + r < t_hi && c * 8 < d;
      const bf16* row = base + static_cast<long long>(t0 + r) * P.ldp + c * 8;
      if (FULL) lc_cp16(q + lc_at<QROW>(r, c), ok ? row + h * d : base, ok);
      lc_cp16(k + lc_at<QROW>(r, c), ok ? row + (H + h) * d : base, ok);
    }
    for (int i = tid; i < LC_C * (EW * 2); i += THREADS) {
      const int r = i / (EW * 2), c = i % (EW * 2);
      const bool ok = t0 + r < t_hi && c < vw;
      lc_cp16(v + lc_at<VROW>(r, c), ok ? base + static_cast<long long>(t0 + r) * P.ldp + 2 * H * d + static_cast<long long>(h) * e + c0 + c * 8 : base, ok);
    }
    asm volatile("cp.async.commit_group;");
  };
  load(0, t_lo);

  // ---- S^T accumulators: tile j covers d columns [8j, + 8); element (e0 + er (+ 8), 8j + kc (+ 1))
  float S[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.f;
  auto each = [&](auto fn) {                         // fn(element, offset inside [d, e]) over this thread's valid elements
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int dd = j * 8 + kc + (i & 1), ee = e0 + er + (i >> 1) * 8;
        if (dd < d && ee < e) fn(S[j][i], static_cast<long long>(dd) * e + ee);
      }
  };
  if (FULL) {
    if (have && P.fresh != nullptr && P.fresh[b] == 0) each([&](float& v, long long at) { v = slot[at]; });
    const float fold = powf(lam, static_cast<float>(seg_len));
    for (int g = 0; g < seg; ++g) {                  // the segments before this one
      const float* loc = local + ((static_cast<long long>(b) * (nseg - 1) + g) * H + h) * static_cast<long long>(d) * e;
      each([&](float& v, long long at) { v = fold * v + loc[at]; });
    }
  }
  int st = 0;
  for (int t0 = t_lo; t0 < t_hi; t0 += LC_C, st ^= 1) {
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();                                 // A: the chunk is in shared memory; everything of the last one has been read
    if (t0 + LC_C < t_hi) load(st ^ 1, t0 + LC_C);
    const uint32_t uq = lc_smem(smem + st * L::STAGE), uk = uq + L::QB, uv = uk + L::QB, uP = lc_smem(smem + L::OFF_P);
    const int n = min(LC_C, t_hi - t0);
    if (FULL) {
      // ---- weighted scores: the 16 x 16 blocks on and under the diagonal, dealt out to the warps
      for (int blk = warp; blk < 10; blk += EW) {
        const int tb = blk < 1 ? 0 : blk < 3 ? 1 : blk < 6 ? 2 : 3, sb = blk - tb * (tb + 1) / 2;
        float acc[2][4] = {};
#pragma unroll
        for (int kk = 0; kk < KS; ++kk) {
          uint32_t fa[4], fb[4];
          lc_ldsm(fa, uq + lc_at<QROW>(tb * 16 + (mi & 1) * 8 + r8, kk * 2 + (mi >> 1)));
          lc_ldsm(fb, uk + lc_at<QROW>(sb * 16 + (mi >> 1) * 8 + r8, kk * 2 + (mi & 1)));
          lc_mma(acc[0], fa, fb[0], fb[1]);
          lc_mma(acc[1], fa, fb[2], fb[3]);
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int t = tb * 16 + er + half * 8;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int s = sb * 16 + j * 8 + kc;
            const float x0 = s <= t ? acc[j][half * 2] * dec[t - s] : 0.f, x1 = s + 1 <= t ? acc[j][half * 2 + 1] * dec[t - s - 1] : 0.f;
            uint32_t hi, lo;
            lc_split(x0, x1, hi, lo);
            const uint32_t at = lc_at<PROW>(t, sb * 2 + j) + kc * 2;
            *reinterpret_cast<uint32_t*>(smem + L::OFF_P + at) = hi;
            *reinterpret_cast<uint32_t*>(smem + L::OFF_P + LC_C * PROW + at) = lo;
          }
        }
      }
      // ---- outputs, 32 tokens at a time: what the state holds (before the barrier for the first half), then the chunk's own tokens
#pragma unroll
      for (int mh = 0; mh < 2; ++mh) {
        float o[2][2][4] = {};
#pragma unroll
        for (int kk = 0; kk < KS; ++kk) {
          uint32_t h0, l0, h1, l1, h2, l2, h3, l3;
          lc_split(S[2 * kk][0], S[2 * kk][1], h0, l0);
          lc_split(S[2 * kk + 1][0], S[2 * kk + 1][1], h1, l1);
          lc_split(S[2 * kk][2], S[2 * kk][3], h2, l2);
          lc_split(S[2 * kk + 1][2], S[2 * kk + 1][3], h3, l3);
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            uint32_t fa[4];
            lc_ldsm(fa, uq + lc_at<QROW>(mh * 32 + m * 16 + (mi & 1) * 8 + r8, kk * 2 + (mi >> 1)));
            lc_mma(o[m][0], fa, h0, h1);
            lc_mma(o[m][1], fa, h2, h3);
            lc_mma(o[m][0], fa, l0, l1);
            lc_mma(o[m][1], fa, l2, l3);
          }
        }
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float f = dec[mh * 32 + m * 16 + (i >> 1) * 8 + er + 1];
            o[m][0][i] *= f;
            o[m][1][i] *= f;
          }
        if (mh == 0) __syncthreads();                // B: scores
#pragma unroll
        for (int kk = 0; kk < 2 + 2 * mh; ++kk) {
          uint32_t fv[4];
          lc_ldsm_t(fv, uv + lc_at<VROW>(kk * 16 + (mi & 1) * 8 + r8, warp * 2 + (mi >> 1)));
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            if (kk > mh * 2 + m) continue;           // above the diagonal
#pragma unroll
            for (int term = 0; term < 2; ++term) {
              uint32_t fa[4];
              lc_ldsm(fa, uP + term * (LC_C * PROW) + lc_at<PROW>(mh * 32 + m * 16 + (mi & 1) * 8 + r8, kk * 2 + (mi >> 1)));
              lc_mma(o[m][0], fa, fv[0], fv[1]);
              lc_mma(o[m][1], fa, fv[2], fv[3]);
            }
          }
        }
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int t = mh * 32 + m * 16 + half * 8 + er;
            bf16* dst = reinterpret_cast<bf16*>(P.out) + static_cast<long long>(s0 + t0 + t) * P.ldo + static_cast<long long>(h) * e + e0 + kc;
#pragma unroll
            for (int j = 0; j < 2; ++j)
              if (t < n && e0 + j * 8 + kc < e) *reinterpret_cast<__nv_bfloat162*>(dst + j * 8) = __floats2bfloat162_rn(o[m][j][half * 2], o[m][j][half * 2 + 1]);
          }
      }
    }
    // ---- state update: S^T = l^n S^T + (w v)^T k, w_s = l^(n - 1 - s)
    const float decC = dec[n];
#pragma unroll
    for (int j = 0; j < NT; ++j) { S[j][0] *= decC; S[j][1] *= decC; S[j][2] *= decC; S[j][3] *= decC; }
#pragma unroll
    for (int kk = 0; kk < LC_C / 16; ++kk) {
      uint32_t fv[4], hi[4], lo[4];
      // (w v)^T as A: rows = v columns, k = tokens; registers {e0 s0, e8 s0, e0 s8, e8 s8}
      lc_ldsm_t(fv, uv + lc_at<VROW>(kk * 16 + (mi >> 1) * 8 + r8, warp * 2 + (mi & 1)));
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int s = n - 1 - (kk * 16 + (i >> 1) * 8 + kc);          // rows behind the portion are zero
        lc_split(__uint_as_float(fv[i] << 16) * dec[max(s, 0)], __uint_as_float(fv[i] & 0xffff0000u) * dec[max(s - 1, 0)], hi[i], lo[i]);
      }
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) {
        uint32_t fk[4];
        lc_ldsm_t(fk, uk + lc_at<QROW>(kk * 16 + (mi & 1) * 8 + r8, j * 2 + (mi >> 1)));
        lc_mma(S[2 * j], hi, fk[0], fk[1]);
        lc_mma(S[2 * j + 1], hi, fk[2], fk[3]);
        lc_mma(S[2 * j], lo, fk[0], fk[1]);
        lc_mma(S[2 * j + 1], lo, fk[2], fk[3]);
      }
    }
  }
  // ---- final state of the sequence, or this segment's own state
  if (!FULL) {
    float* loc = local + ((static_cast<long long>(b) * (nseg - 1) + seg) * H + h) * static_cast<long long>(d) * e;
    each([&](float& v, long long at) { loc[at] = v; });
  } else if (have && t_hi == len) {
    each([&](float& v, long long at) { slot[at] = v; });
  }
}

template <int DP, int EW>
static int lc_launch(const VbLightning& p, int nseg, float* local, cudaStream_t s) {
  const dim3 grid((p.e + EW * 16 - 1) / (EW * 16), p.H, p.B * nseg);
  auto go = [&](auto kern) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LcSmem<DP, EW>::TOTAL);
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<grid, 32 * EW, LcSmem<DP, EW>::TOTAL, s>>>(p, nseg, local);
    return static_cast<int>(cudaGetLastError());
  };
  const int rc = nseg > 1 ? go(lightning_chunk_kernel<DP, EW, false>) : 0;
  return rc == 0 ? go(lightning_chunk_kernel<DP, EW, true>) : rc;
}

}  // namespace vb

using namespace vb;

// Segments a sequence is cut into (1 = none; the workspace then needs B * (nseg - 1) * H * d * e floats), or 0 when the sizes are not
// served. all_fresh: every sequence starts from zero (a segment may not read a stored state that another one replaces).
extern "C" int vb_lightning_chunk_segments(int T, int B, int H, int d, int e, int all_fresh) {
  if (d % 8 || e % 8 || d > 256 || d < 8 || e < 8 || B > 65535 || H > 65535) return 0;
  if (!all_fresh) return 1;
  const int cols = d > 128 && e <= 64 ? 64 : 128, ctas = B * H * ((e + cols - 1) / cols);
  int s = 148 / ctas;
  const int by_len = T / B / (4 * LC_C);
  if (s > by_len) s = by_len;
  if (s > 32) s = 32;
  return (s < 1 || static_cast<long long>(B) * s > 65535) ? 1 : s;
}

extern "C" int vb_lightning_chunk(const VbLightning* p, int nseg, float* local, cudaStream_t s) {
  if (p->ldp % 8 || (reinterpret_cast<uintptr_t>(p->p) & 15) || (p->ldo % 2) || (reinterpret_cast<uintptr_t>(p->out) & 3)) return -1;
  return p->e <= 64 ? lc_launch<256, 4>(*p, nseg, local, s) : lc_launch<256, 8>(*p, nseg, local, s);
}
