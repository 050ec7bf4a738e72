// Generalized delta rule over prompts, 16 tokens at a time (bf16 rows, fp32 state, head size <= 128).
//
//   S_t = diag(w_t) S_(t-1) - (a_t u_t)(u_t^T S_(t-1)) + k_t v_t^T,   o_t = S_t^T r_t
//
// Inside a chunk, with W_t the product of its decays up to t, let U_t = u_t W_(t-1), R_t = r_t W_t, B_t = -a_t u_t / W_t, K_t = k_t / W_t (a decay
// is at least exp(-exp(-1/2)), so 16 of them stay far from the ends of the fp32 range), and y_t = u_t^T S_(t-1). Then
//   Y = X S_0 + Z V      with T = (I - tril(U B^T, -1))^-1, X = T U, Z = T tril(U K^T, -1)
//   O = R S_0 + tril(R B^T) Y + tril(R K^T) V
//   S = diag(W_16) (S_0 + B^T Y + K^T V)
// One CTA = (sequence segment, head). Producer warps own a stage of the shared-memory ring each and form a chunk's X, Z, R, B, K and score
// matrices, which do not depend on the state (T by forward substitution in fp32). State warps own 16 columns of v each: S^T is an fp32
// accumulator in registers for the whole segment, and its fragments as accumulator and as A operand of the next chunk are the same
// registers, as are those of Y^T; no state warp waits for another. The matrices are 16 tokens high, too low for the 128-row
// tiles of tcgen05, hence m16n8k16. Every fp32 value that enters a product is split into two bf16 terms (products high x high, high x low,
// low x high).
//
// Few long prompts are cut into segments. A segment acts on the state as S -> M S + N; a first launch computes M (from the identity,
// without values) and N (from zero) of every segment but the last, a second folds them into the segments' starting states, the
// third is the whole.
#include "mixers.h"
#include "mixer_common.cuh"
#include "tcgen05_common.cuh"

#include <math.h>

namespace vb {

typedef __nv_bfloat16 bf16;
constexpr int DC_C = 16, DC_SQ = 16 * 48;            // tokens of a chunk; bytes of a 16 x 16 bf16 tile (rows of 48 bytes: shifted banks)

template <int DP, int PW>
struct DcSmem {
  static constexpr int PITCH = DP * 2 + 16, OPER = DC_C * PITCH;
  // operands [token][channel]: high and low terms of X (first U), R, B, K, then v
  static constexpr int X = 0, R = 2 * OPER, B = 4 * OPER, K = 6 * OPER, V = 8 * OPER;
  static constexpr int Z = 9 * OPER, RK = Z + 2 * DC_SQ, RB = RK + 2 * DC_SQ, W = RB + 2 * DC_SQ;   // score tiles [t][s], W_16
  static constexpr int STAGE = W + DP * 4, BARS = PW * STAGE, TOTAL = BARS + PW * 16;
};

__device__ int g_delta_chunk_status[1];

__device__ __forceinline__ void dc_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void dc_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void dc_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t dc_transpose(uint32_t x) {
  uint32_t y;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
  return y;
}
// two floats as a bf16 pair plus the pair of what rounding dropped
__device__ __forceinline__ void dc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}
// d += (ah + al)(bh + bl) without the product of the low terms
__device__ __forceinline__ void dc_mma3(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
  dc_mma(d, ah, bl0, bl1);
  dc_mma(d, al, bh0, bh1);
  dc_mma(d, ah, bh0, bh1);
}
__device__ __forceinline__ float dc_sigmoid(float z) { return __fdividef(1.f, 1.f + exp2f(-1.4426950408889634f * z)); }
__device__ __forceinline__ float dc_low(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float dc_high(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }
__device__ __forceinline__ void dc_put(uint8_t* p, uint32_t v) { *reinterpret_cast<uint32_t*>(p) = v; }

// A 16 x 16 tile in accumulator form (two n8 tiles) -> high and low terms in shared memory; strict: without the diagonal, else with it;
// entries above are zero.
__device__ __forceinline__ void dc_store_lower(uint8_t* tile, const float (&c)[2][4], int lane, bool strict) {
  const int g = lane >> 2, q = (lane & 3) * 2;
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = g + half * 8, s = n * 8 + q;
      const float x = s < t || (!strict && s == t) ? c[n][half * 2] : 0.f, y = s + 1 < t || (!strict && s + 1 == t) ? c[n][half * 2 + 1] : 0.f;
      uint32_t hi, lo;
      dc_split(x, y, hi, lo);
      dc_put(tile + t * 48 + s * 2, hi);
      dc_put(tile + DC_SQ + t * 48 + s * 2, lo);
    }
}

template <int DP, int PW, bool FULL>
__global__ void __launch_bounds__((DP / 16 + PW) * 32, DP <= 64 && PW == 4 ? 2 : 1)
delta_chunk_kernel(const VbDelta P, int nseg, float* __restrict__ ws, int* status) {
  using L = DcSmem<DP, PW>;
  constexpr int SW = DP / 16, NP = (DP + 63) / 64;
  extern __shared__ __align__(16) uint8_t smem[];
  uint64_t *full = reinterpret_cast<uint64_t*>(smem + L::BARS), *empty = full + PW;

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mi = lane >> 3, r8 = lane & 7;
  const int h = blockIdx.x, part = FULL ? 0 : blockIdx.z & 1, seg = FULL ? blockIdx.z : blockIdx.z >> 1, b = blockIdx.y;   // part 1: M
  const int d = P.d, H = P.H, W = H * d, s0 = P.cu[b], len = P.cu[b + 1] - s0;
  const int seg_len = ((len + nseg - 1) / nseg + DC_C - 1) / DC_C * DC_C;
  const int t_lo = seg * seg_len, t_hi = min(len, t_lo + seg_len);
  if (t_lo >= t_hi) return;                          // uniform over the CTA
  if (!FULL && t_hi == len) return;                  // nothing follows
  const int nch = (t_hi - t_lo + DC_C - 1) / DC_C;
  const bool values = part == 0;

  if (tid == 0) {
    for (int i = 0; i < PW; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], SW);
    }
    mbar_fence_init();
  }
  __syncthreads();

  const long long size = static_cast<long long>(d) * d;
  float* own = ws != nullptr ? ws + (((static_cast<long long>(b) * nseg + seg) * H + h) * 2 + part) * size : nullptr;
  bool ok = true;
  if (warp < SW) {
    // ------------------------------------------------------------------ state: rows 16 warp .. of S^T
    const int g = lane >> 2, q = (lane & 3) * 2, e0 = warp * 16;
    const bool have = FULL && P.slots != nullptr && P.slots[b] >= 0;
    float* slot = have ? P.state + static_cast<long long>(P.slots[b]) * P.slot_stride + h * size : nullptr;
    const float* src = !FULL ? nullptr : nseg > 1 ? own : (have && !(P.fresh != nullptr && P.fresh[b] != 0) ? slot : nullptr);
    float S[2 * SW][4];
#pragma unroll
    for (int j = 0; j < 2 * SW; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int c = j * 8 + q + (i & 1), e = e0 + g + (i >> 1) * 8;
        S[j][i] = part == 1 ? (c == e && c < d ? 1.f : 0.f) : (src != nullptr && c < d && e < d ? src[static_cast<long long>(c) * d + e] : 0.f);
      }
    bf16* out = reinterpret_cast<bf16*>(P.out) + static_cast<long long>(s0 + t_lo) * P.ldo + static_cast<long long>(h) * d;
    // row and column of this lane's ldmatrix row: tokens x channels as B operand [n][k], as B operand [k][n] (transposed), as A operand [k][m] (transposed)
    const uint32_t at_n = ((mi >> 1) * 8 + r8) * L::PITCH + (mi & 1) * 16, at_k = ((mi & 1) * 8 + r8) * L::PITCH + (mi >> 1) * 16;
    const uint32_t at_v = ((mi >> 1) * 8 + r8) * L::PITCH + (e0 + (mi & 1) * 8) * 2, at_sq = ((mi >> 1) * 8 + r8) * 48 + (mi & 1) * 16;
    for (int j = 0; j < nch; ++j) {
      const int st = j % PW;
      uint8_t* stage = smem + st * L::STAGE;
      const uint32_t base = smem_u32(stage);
      if (!__all_sync(0xffffffffu, mbar_wait(&full[st], (j / PW) & 1))) { ok = false; break; }
      float Y[2][4] = {}, O[2][4] = {};
#pragma unroll
      for (int k = 0; k < SW; ++k) {
        uint32_t sh[4], sl[4], xh[4], xl[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) dc_split(S[2 * k + (i >> 1)][(i & 1) * 2], S[2 * k + (i >> 1)][(i & 1) * 2 + 1], sh[i], sl[i]);
        dc_ldsm(xh, base + L::X + at_n + k * 32);
        dc_ldsm(xl, base + L::X + L::OPER + at_n + k * 32);
        dc_mma3(Y[0], sh, sl, xh[0], xh[1], xl[0], xl[1]);
        dc_mma3(Y[1], sh, sl, xh[2], xh[3], xl[2], xl[3]);
        if (FULL) {
          dc_ldsm(xh, base + L::R + at_n + k * 32);
          dc_ldsm(xl, base + L::R + L::OPER + at_n + k * 32);
          dc_mma3(O[0], sh, sl, xh[0], xh[1], xl[0], xl[1]);
          dc_mma3(O[1], sh, sl, xh[2], xh[3], xl[2], xl[3]);
        }
      }
      uint32_t v[4], zh[4], zl[4], yh[4], yl[4];
      if (values) {
        dc_ldsm_t(v, base + L::V + at_v);
        dc_ldsm(zh, base + L::Z + at_sq);
        dc_ldsm(zl, base + L::Z + DC_SQ + at_sq);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          dc_mma(Y[n], v, zl[2 * n], zl[2 * n + 1]);
          dc_mma(Y[n], v, zh[2 * n], zh[2 * n + 1]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) dc_split(Y[i >> 1][(i & 1) * 2], Y[i >> 1][(i & 1) * 2 + 1], yh[i], yl[i]);
#pragma unroll
      for (int k = 0; k < SW; ++k) {
        uint32_t bh[4], bl[4];
        dc_ldsm_t(bh, base + L::B + at_k + k * 32);
        dc_ldsm_t(bl, base + L::B + L::OPER + at_k + k * 32);
        dc_mma3(S[2 * k], yh, yl, bh[0], bh[1], bl[0], bl[1]);
        dc_mma3(S[2 * k + 1], yh, yl, bh[2], bh[3], bl[2], bl[3]);
        if (values) {
          dc_ldsm_t(bh, base + L::K + at_k + k * 32);
          dc_ldsm_t(bl, base + L::K + L::OPER + at_k + k * 32);
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            dc_mma(S[2 * k + n], v, bl[2 * n], bl[2 * n + 1]);
            dc_mma(S[2 * k + n], v, bh[2 * n], bh[2 * n + 1]);
          }
        }
      }
      const float* wc = reinterpret_cast<const float*>(stage + L::W);
#pragma unroll
      for (int k = 0; k < 2 * SW; ++k) {
        const float2 w = *reinterpret_cast<const float2*>(wc + k * 8 + q);
        S[k][0] *= w.x; S[k][1] *= w.y; S[k][2] *= w.x; S[k][3] *= w.y;
      }
      if (FULL) {
        dc_ldsm(zh, base + L::RK + at_sq);
        dc_ldsm(zl, base + L::RK + DC_SQ + at_sq);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          dc_mma(O[n], v, zl[2 * n], zl[2 * n + 1]);
          dc_mma(O[n], v, zh[2 * n], zh[2 * n + 1]);
        }
        dc_ldsm(zh, base + L::RB + at_sq);
        dc_ldsm(zl, base + L::RB + DC_SQ + at_sq);
#pragma unroll
        for (int n = 0; n < 2; ++n) dc_mma3(O[n], yh, yl, zh[2 * n], zh[2 * n + 1], zl[2 * n], zl[2 * n + 1]);
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty[st]);
      if (FULL) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          // [e, t] -> [t, e]: this lane's token, two pairs of columns
          const uint32_t lo8 = dc_transpose(pack_bf16x2(O[n][0], O[n][1])), hi8 = dc_transpose(pack_bf16x2(O[n][2], O[n][3]));
          const int t = j * DC_C + n * 8 + g;
          if (t_lo + t < t_hi) {
            bf16* dst = out + static_cast<long long>(t) * P.ldo + e0 + q;
            if (e0 + q < d) *reinterpret_cast<uint32_t*>(dst) = lo8;
            if (e0 + 8 + q < d) *reinterpret_cast<uint32_t*>(dst + 8) = hi8;
          }
        }
      }
    }
    float* dst = FULL ? (t_hi == len ? slot : nullptr) : own;
    if (ok && dst != nullptr) {
#pragma unroll
      for (int j = 0; j < 2 * SW; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int c = j * 8 + q + (i & 1), e = e0 + g + (i >> 1) * 8;
          if (c < d && e < d) dst[static_cast<long long>(c) * d + e] = S[j][i];
        }
    }
  } else {
    // ------------------------------------------------------------------ producers: chunks pw, pw + PW, ...; the stage is theirs
    const int pw = warp - SW;
    uint8_t* stage = smem + pw * L::STAGE;
    const uint32_t base = smem_u32(stage);
    const bf16 *prow = reinterpret_cast<const bf16*>(P.p) + static_cast<long long>(s0) * P.ldp + h * d, *zrow = reinterpret_cast<const bf16*>(P.zw) + static_cast<long long>(s0) * P.ldz + h * d;
    const int g = lane >> 2, q = (lane & 3) * 2;
    float w0[NP][2], ab[NP][2];
    bool on[NP];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int c = i * 64 + lane * 2;
      on[i] = c < d;
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        w0[i][x] = on[i] ? __bfloat162float(reinterpret_cast<const bf16*>(P.w0)[h * d + c + x]) : 0.f;
        ab[i][x] = on[i] ? __bfloat162float(reinterpret_cast<const bf16*>(P.ab)[h * d + c + x]) : 0.f;
      }
    }
    for (int j = pw; j < nch; j += PW) {
      const int t0 = t_lo + j * DC_C, n = min(DC_C, t_hi - t0);   // live tokens
      auto fetch = [&](const bf16* p, long long ld, int i, int t) {
        return on[i] && t < n ? *reinterpret_cast<const uint32_t*>(p + static_cast<long long>(t0 + t) * ld + i * 64 + lane * 2) : 0u;
      };
      uint32_t rk[NP][DC_C], rz[DC_C], ra[DC_C];
      float ss[DC_C];
#pragma unroll
      for (int i = 0; i < NP; ++i)
#pragma unroll
        for (int t = 0; t < DC_C; ++t) rk[i][t] = fetch(prow + W, P.ldp, i, t);
#pragma unroll
      for (int t = 0; t < DC_C; ++t) rz[t] = fetch(zrow, P.ldz, 0, t);
#pragma unroll
      for (int t = 0; t < DC_C; ++t) ra[t] = fetch(prow + 3 * W, P.ldp, 0, t);
#pragma unroll
      for (int t = 0; t < DC_C; ++t) {
        ss[t] = 0.f;
#pragma unroll
        for (int i = 0; i < NP; ++i) ss[t] += dc_low(rk[i][t]) * dc_low(rk[i][t]) + dc_high(rk[i][t]) * dc_high(rk[i][t]);
      }
      // sums over the lanes, 16 tokens at once: each step halves the tokens a lane is in charge of
#pragma unroll
      for (int m = 8; m >= 1; m >>= 1) {
        const bool up = (lane & (2 * m)) != 0;
#pragma unroll
        for (int i = 0; i < m; ++i) {
          const float give = up ? ss[i] : ss[i + m], keep = up ? ss[i + m] : ss[i];
          ss[i] = keep + __shfl_xor_sync(0xffffffffu, give, 2 * m);
        }
      }
      const float own_u = rsqrtf(ss[0] + __shfl_xor_sync(0xffffffffu, ss[0], 1) + 1e-6f);   // of token lane / 2
      float iu[DC_C];
#pragma unroll
      for (int t = 0; t < DC_C; ++t) iu[t] = __shfl_sync(0xffffffffu, own_u, 2 * t);
      if (j >= PW && !__all_sync(0xffffffffu, mbar_wait(&empty[pw], ((j / PW) & 1) ^ 1))) { ok = false; break; }
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int c = i * 64 + lane * 2;
        if (i > 0) {
#pragma unroll
          for (int t = 0; t < DC_C; ++t) rz[t] = fetch(zrow, P.ldz, i, t);
#pragma unroll
          for (int t = 0; t < DC_C; ++t) ra[t] = fetch(prow + 3 * W, P.ldp, i, t);
        }
        uint32_t rr[DC_C];
        if (FULL) {
#pragma unroll
          for (int t = 0; t < DC_C; ++t) rr[t] = fetch(prow, P.ldp, i, t);
        }
        if (c < DP) {
          if (values) {
#pragma unroll
            for (int t = 0; t < DC_C; ++t) dc_put(stage + L::V + t * L::PITCH + c * 2, fetch(prow + 2 * W, P.ldp, i, t));
          }
          float D0 = 1.f, D1 = 1.f;                  // product of the decays
#pragma unroll
          for (int t = 0; t < DC_C; ++t) {
            const bool live = t < n;
            const float k0 = dc_low(rk[i][t]), k1 = dc_high(rk[i][t]), u0 = k0 * iu[t], u1 = k1 * iu[t];
            uint32_t hi, lo;
            uint8_t* at = stage + t * L::PITCH + c * 2;
            dc_split(u0 * D0, u1 * D1, hi, lo);
            dc_put(at + L::X, hi);
            dc_put(at + L::X + L::OPER, lo);
            // -exp(-1/2) log2(e) = -0.87503...
            constexpr float fall = -0.60653065971263342f * 1.4426950408889634f;
            if (live) {
              D0 *= exp2f(fall * dc_sigmoid(dc_low(rz[t]) + w0[i][0]));
              D1 *= exp2f(fall * dc_sigmoid(dc_high(rz[t]) + w0[i][1]));
            }
            const float i0 = __fdividef(1.f, D0), i1 = __fdividef(1.f, D1);
            dc_split(-dc_sigmoid(dc_low(ra[t]) + ab[i][0]) * u0 * i0, -dc_sigmoid(dc_high(ra[t]) + ab[i][1]) * u1 * i1, hi, lo);
            dc_put(at + L::B, hi);
            dc_put(at + L::B + L::OPER, lo);
            dc_split(k0 * i0, k1 * i1, hi, lo);
            dc_put(at + L::K, hi);
            dc_put(at + L::K + L::OPER, lo);
            if (FULL) {
              dc_split(dc_low(rr[t]) * D0, dc_high(rr[t]) * D1, hi, lo);
              dc_put(at + L::R, hi);
              dc_put(at + L::R + L::OPER, lo);
            }
          }
          *reinterpret_cast<float2*>(stage + L::W + c * 4) = make_float2(D0, D1);
        }
        __syncwarp();
      }
      // ---- scores
      const uint32_t at_m = ((mi & 1) * 8 + r8) * L::PITCH + (mi >> 1) * 16;   // A operand [m][k]
      const uint32_t at_n = ((mi >> 1) * 8 + r8) * L::PITCH + (mi & 1) * 16;   // B operand [n][k]
      float ub[2][4] = {}, uk[2][4] = {}, rb[2][4] = {}, rkk[2][4] = {};
#pragma unroll
      for (int k = 0; k < SW; ++k) {
        uint32_t uh[4], ul[4], rh[4], rl[4], xh[4], xl[4];
        dc_ldsm(uh, base + L::X + at_m + k * 32);
        dc_ldsm(ul, base + L::X + L::OPER + at_m + k * 32);
        if (FULL) {
          dc_ldsm(rh, base + L::R + at_m + k * 32);
          dc_ldsm(rl, base + L::R + L::OPER + at_m + k * 32);
        }
        dc_ldsm(xh, base + L::B + at_n + k * 32);
        dc_ldsm(xl, base + L::B + L::OPER + at_n + k * 32);
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          dc_mma3(ub[m], uh, ul, xh[2 * m], xh[2 * m + 1], xl[2 * m], xl[2 * m + 1]);
          if (FULL) dc_mma3(rb[m], rh, rl, xh[2 * m], xh[2 * m + 1], xl[2 * m], xl[2 * m + 1]);
        }
        if (values) {
          dc_ldsm(xh, base + L::K + at_n + k * 32);
          dc_ldsm(xl, base + L::K + L::OPER + at_n + k * 32);
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            dc_mma3(uk[m], uh, ul, xh[2 * m], xh[2 * m + 1], xl[2 * m], xl[2 * m + 1]);
            if (FULL) dc_mma3(rkk[m], rh, rl, xh[2 * m], xh[2 * m + 1], xl[2 * m], xl[2 * m + 1]);
          }
        }
      }
      // ---- T = (I - tril(U B^T, -1))^-1: a lane solves for a column. The tile of scores passes through the place of RB, T through that of RK
      float* sn = reinterpret_cast<float*>(stage + L::RB);                     // [16][20]
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        *reinterpret_cast<float2*>(sn + g * 20 + m * 8 + q) = make_float2(ub[m][0], ub[m][1]);
        *reinterpret_cast<float2*>(sn + (g + 8) * 20 + m * 8 + q) = make_float2(ub[m][2], ub[m][3]);
      }
      if (values) dc_store_lower(stage + L::Z, uk, lane, true);
      __syncwarp();
      {
        const int col = lane & 15;
        float x[DC_C];
#pragma unroll
        for (int t = 0; t < DC_C; ++t) {
          float a0 = t == col ? 1.f : 0.f, a1 = 0.f;
#pragma unroll
          for (int s = 0; s < t; s += 4) {
            const float4 m4 = *reinterpret_cast<const float4*>(sn + t * 20 + s);
            a0 = fmaf(m4.x, x[s], a0);
            if (s + 1 < t) a1 = fmaf(m4.y, x[s + 1], a1);
            if (s + 2 < t) a0 = fmaf(m4.z, x[s + 2], a0);
            if (s + 3 < t) a1 = fmaf(m4.w, x[s + 3], a1);
          }
          x[t] = a0 + a1;                             // zero above the diagonal
        }
        if (lane < 16) {
#pragma unroll
          for (int t = 0; t < DC_C; ++t) {
            const bf16 hi = __float2bfloat16(x[t]);
            reinterpret_cast<bf16*>(stage + L::RK + t * 48)[col] = hi;
            reinterpret_cast<bf16*>(stage + L::RK + DC_SQ + t * 48)[col] = __float2bfloat16(x[t] - __bfloat162float(hi));
          }
        }
      }
      __syncwarp();
      uint32_t th[4], tl[4];
      const uint32_t sq_m = ((mi & 1) * 8 + r8) * 48 + (mi >> 1) * 16;         // A operand [m][k], and B operand [k][n] (transposed)
      dc_ldsm(th, base + L::RK + sq_m);
      dc_ldsm(tl, base + L::RK + DC_SQ + sq_m);
      // ---- X = T U in U's place, 16 channels at a time
#pragma unroll
      for (int k = 0; k < SW; ++k) {
        uint32_t xh[4], xl[4];
        float x[2][4] = {};
        dc_ldsm_t(xh, base + L::X + at_m + k * 32);
        dc_ldsm_t(xl, base + L::X + L::OPER + at_m + k * 32);
#pragma unroll
        for (int m = 0; m < 2; ++m) dc_mma3(x[m], th, tl, xh[2 * m], xh[2 * m + 1], xl[2 * m], xl[2 * m + 1]);
        __syncwarp();
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            uint32_t hi, lo;
            dc_split(x[m][half * 2], x[m][half * 2 + 1], hi, lo);
            uint8_t* at = stage + L::X + (g + half * 8) * L::PITCH + (k * 16 + m * 8 + q) * 2;
            dc_put(at, hi);
            dc_put(at + L::OPER, lo);
          }
      }
      // ---- Z = T tril(U K^T, -1)
      if (values) {
        uint32_t xh[4], xl[4];
        float z[2][4] = {};
        dc_ldsm_t(xh, base + L::Z + sq_m);
        dc_ldsm_t(xl, base + L::Z + DC_SQ + sq_m);
#pragma unroll
        for (int m = 0; m < 2; ++m) dc_mma3(z[m], th, tl, xh[2 * m], xh[2 * m + 1], xl[2 * m], xl[2 * m + 1]);
        __syncwarp();
        dc_store_lower(stage + L::Z, z, lane, true);
      }
      __syncwarp();
      if (FULL) {
        dc_store_lower(stage + L::RK, rkk, lane, false);
        dc_store_lower(stage + L::RB, rb, lane, false);
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&full[pw]);
    }
  }
  if (!ok && lane == 0) atomicExch(status, ST_TIMEOUT_PRODUCER);
}

// Starting states of the segments: S_(g+1) = M_g S_g + N_g, in N's place. One CTA per (sequence, head, 32 columns of v).
__global__ void __launch_bounds__(256)
delta_fold_kernel(const VbDelta P, int nseg, float* __restrict__ ws) {
  extern __shared__ float sm[];                      // [d][32], two of them
  const int h = blockIdx.x, b = blockIdx.y, c0 = blockIdx.z * 32, d = P.d, col = threadIdx.x & 31, rg = threadIdx.x >> 5;
  const int len = P.cu[b + 1] - P.cu[b], seg_len = ((len + nseg - 1) / nseg + DC_C - 1) / DC_C * DC_C;
  const long long size = static_cast<long long>(d) * d;
  const bool c_ok = c0 + col < d, have = P.slots != nullptr && P.slots[b] >= 0 && !(P.fresh != nullptr && P.fresh[b] != 0);
  float *cur = sm, *nxt = sm + d * 32;
  const float* st = have ? P.state + static_cast<long long>(P.slots[b]) * P.slot_stride + h * size : nullptr;
  for (int r = rg; r < d; r += 8) cur[r * 32 + col] = st != nullptr && c_ok ? st[static_cast<long long>(r) * d + c0 + col] : 0.f;
  __syncthreads();
  for (int g = 0; g < nseg && g * seg_len < len; ++g) {
    float *N = ws + ((static_cast<long long>(b) * nseg + g) * P.H + h) * 2 * size, *M = N + size;
    const bool last = (g + 1) * seg_len >= len;
    for (int r = rg; r < d; r += 8) {
      if (!last) {
        float a = c_ok ? N[static_cast<long long>(r) * d + c0 + col] : 0.f;
        const float* m = M + static_cast<long long>(r) * d;
        for (int k = 0; k < d; ++k) a = fmaf(m[k], cur[k * 32 + col], a);
        nxt[r * 32 + col] = a;
      }
      if (c_ok) N[static_cast<long long>(r) * d + c0 + col] = cur[r * 32 + col];
    }
    __syncthreads();
    float* t = cur; cur = nxt; nxt = t;
  }
}

}  // namespace vb

using namespace vb;

// Segments that the prompts are cut into (1: not cut; 0: sizes that the chunked kernel does not serve).
extern "C" int vb_delta_chunk_segments(const VbDelta* p) {
  if (p->d > 128 || p->d % 2 || p->d < 2) return 0;
  const long long ctas = static_cast<long long>(p->B) * p->H;
  if (ctas <= 0) return 1;
  // M and N of all segments but the last make two CTAs each; about as many as run at once
  const long long room = num_sms() * (p->d <= 64 ? 2 : 1);
  long long n = 1 + room / (2 * ctas), most = p->T / p->B / 512;
  if (n > most) n = most;
  if (n > 32) n = 32;
  return n < 4 ? 1 : static_cast<int>(n);
}

// nseg > 1: ws holds B nseg H 2 d d floats. Returns -1 for alignments it does not serve.
extern "C" int vb_delta_chunk(const VbDelta* p, int nseg, float* ws, cudaStream_t s) {
  auto mis = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 3) != 0; };
  if (p->ldp % 2 || p->ldz % 2 || p->ldo % 2 || mis(p->p) || mis(p->zw) || mis(p->out) || p->B > 65535 || nseg < 1 || nseg > 32) return -1;
  static int* status = nullptr;
  if (status == nullptr) cudaGetSymbolAddress(reinterpret_cast<void**>(&status), g_delta_chunk_status);
  auto go = [&](auto kern, int threads, int smem, bool whole) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<dim3(p->H, p->B, whole ? nseg : 2 * (nseg - 1)), threads, smem, s>>>(*p, nseg, ws, status);
    return static_cast<int>(cudaGetLastError());
  };
#define VB_DC(DP_, PW_, FULL_) go(delta_chunk_kernel<DP_, PW_, FULL_>, (DP_ / 16 + PW_) * 32, DcSmem<DP_, PW_>::TOTAL, FULL_)
  const bool few = static_cast<long long>(p->B) * p->H * nseg <= num_sms();   // a CTA has an SM for itself
  int rc = 0;
  if (nseg > 1) {
    if (p->d <= 32) rc = VB_DC(32, 4, false);
    else if (p->d <= 64) rc = VB_DC(64, 4, false);
    else if (p->d <= 96) rc = VB_DC(96, 4, false);
    else rc = VB_DC(128, 4, false);
    if (rc != 0) return rc;
    delta_fold_kernel<<<dim3(p->H, p->B, (p->d + 31) / 32), 256, 2 * p->d * 32 * 4, s>>>(*p, nseg, ws);
    rc = static_cast<int>(cudaGetLastError());
    if (rc != 0) return rc;
  }
  if (p->d <= 32) rc = few ? VB_DC(32, 8, true) : VB_DC(32, 4, true);
  else if (p->d <= 64) rc = few ? VB_DC(64, 8, true) : VB_DC(64, 4, true);
  else if (p->d <= 96) rc = few ? VB_DC(96, 6, true) : VB_DC(96, 4, true);
  else rc = VB_DC(128, 4, true);
#undef VB_DC
  return rc;
}

extern "C" int vb_delta_chunk_status() {
  int h = 0;
  if (cudaMemcpyFromSymbol(&h, g_delta_chunk_status, sizeof(int)) != cudaSuccess) return -1;
  if (h != 0) {
    const int z = 0;
    cudaMemcpyToSymbol(g_delta_chunk_status, &z, sizeof(int));
  }
  return h;
}
