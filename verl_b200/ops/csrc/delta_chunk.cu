// Generalized delta rule over prompts, 16 tokens at a time (bf16 rows, fp32 state, head size <= 128).
//
//   S_t = diag(w_t) S_(t-1) - (a_t u_t)(u_t^T S_(t-1)) + k_t v_t^T,   o_t = S_t^T r_t
//
// Inside a chunk, with W_t the product of its decays up to t, let U_t = k_t W_(t-1), R_t = r_t W_t, B_t = -a_t k_t / W_t, K_t = k_t / W_t (a decay
// is at least exp(-exp(-1/2)), so 16 of them stay far from the ends of the fp32 range), D the inverse lengths of the keys (u = D k) and
// y_t = D_t u_t^T S_(t-1). Then
//   Y = X S_0 + Z V      with T = D (I - tril(D U B^T D, -1))^-1 D, X = T U, Z = T tril(U K^T, -1)
//   O = R S_0 + tril(R B^T) Y + tril(R K^T) V
//   S = diag(W_16) (S_0 + B^T Y + K^T V)
// One CTA = (sequence segment, head). Groups of producer warps fill the stages of a shared-memory ring in turn with a chunk's X, Z, R, B, K
// and score matrices, which do not depend on the state: a warp takes 16 channels (a lane two channels of four tokens), then a score matrix
// (the first one also T, by forward substitution in fp32), then 16 channels of X. State warps own 16 columns of v each: S^T is an fp32
// accumulator in registers for the whole segment, and its fragments as accumulator and as A operand of the next chunk are the same
// registers, as are those of Y^T; no state warp waits for another. The matrices are 16 tokens high, too low for the 128-row
// tiles of tcgen05, hence m16n8k16. Every fp32 value that enters the state through a product is split into two bf16 terms (products high x
// high, high x low, low x high); the read-out takes the state in two terms and R, rounded like the output, in one.
//
// Few long prompts are cut into segments. A segment acts on the state as S -> M S + N; a first launch computes M (from the identity,
// without values) and N (from zero) of every segment but the last, a second folds them into the segments' starting states, the
// third is the whole.
#include "mixers.h"
#include "mixer_common.cuh"
#include "tcgen05_common.cuh"

#include <math.h>
#include <type_traits>

namespace vb {

typedef __nv_bfloat16 bf16;
constexpr int DC_C = 16, DC_SQ = 16 * 48;            // tokens of a chunk; bytes of a 16 x 16 bf16 tile (rows of 48 bytes: shifted banks)

template <int DP, int G, int NS>
struct DcSmem {
  static constexpr int PITCH = DP * 2 + 16, OPER = DC_C * PITCH;
  // operands [token][channel]: high and low terms of X (first U), B and K, then R, then v
  static constexpr int X = 0, B = 2 * OPER, K = 4 * OPER, R = 6 * OPER, V = 7 * OPER;
  static constexpr int Z = 8 * OPER, RK = Z + 2 * DC_SQ, RB = RK + DC_SQ, W = RB + DC_SQ;   // score tiles [t][s] (Z: two terms), W_16
  static constexpr int STAGE = W + DP * 4;
  // per group: rows of k, zw, za and r as they come, scores of T [s][t], T in two terms [s][t], partial sums of squares [warp][token], norms of
  // the keys
  static constexpr int N = 4 * OPER, T = N + DC_C * 20 * 4, KK = T + 2 * DC_SQ, IU = KK + DP / 16 * 64, SCRATCH = IU + 64;
  static constexpr int GROUPS = NS * STAGE, BARS = GROUPS + G * SCRATCH, TOTAL = BARS + NS * 16;
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
// two floats as a bf16 pair (cut off) plus the pair of what is missing
__device__ __forceinline__ void dc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const uint32_t a = __float_as_uint(x), b = __float_as_uint(y);
  hi = __byte_perm(a, b, 0x7632);
  lo = pack_bf16x2(x - __uint_as_float(a & 0xffff0000u), y - __uint_as_float(b & 0xffff0000u));
}
// d += (ah + al)(bh + bl) without the product of the low terms, the mixed ones in an accumulator of their own
__device__ __forceinline__ void dc_mma3(float (&d)[4], float (&mixed)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
  dc_mma(d, ah, bh0, bh1);
  dc_mma(mixed, ah, bl0, bl1);
  dc_mma(mixed, al, bh0, bh1);
}
__device__ __forceinline__ float dc_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float dc_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float dc_sigmoid(float z) { return dc_rcp(1.f + dc_ex2(-1.4426950408889634f * z)); }
__device__ __forceinline__ float dc_low(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float dc_high(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }
// 16 bytes from global to shared memory, the first n of them read (0 or 16) and the others zero
__device__ __forceinline__ void dc_fetch16(uint32_t dst, const void* src, uint32_t n) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void dc_put(uint8_t* p, uint32_t v) { *reinterpret_cast<uint32_t*>(p) = v; }
__device__ __forceinline__ void dc_put2(uint8_t* p, int low, float x, float y) {
  uint32_t hi, lo;
  dc_split(x, y, hi, lo);
  dc_put(p, hi);
  dc_put(p + low, lo);
}

// A 16 x 16 tile in accumulator form (two n8 tiles) -> bf16 in shared memory, two terms or one; strict: without the diagonal, else with
// it; entries above are zero.
template <bool TWO>
__device__ __forceinline__ void dc_store_lower(uint8_t* tile, const float (&c)[2][4], int lane, bool strict) {
  const int g = lane >> 2, q = (lane & 3) * 2;
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = g + half * 8, s = n * 8 + q, most = strict ? t - 1 : t;
      const float x = s <= most ? c[n][half * 2] : 0.f, y = s + 1 <= most ? c[n][half * 2 + 1] : 0.f;
      if (TWO) dc_put2(tile + t * 48 + s * 2, DC_SQ, x, y);
      else dc_put(tile + t * 48 + s * 2, pack_bf16x2(x, y));
    }
}

template <int N> __device__ __forceinline__ void dc_more_registers() { asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(N)); }
template <int N> __device__ __forceinline__ void dc_fewer_registers() { asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(N)); }

// Where registers allow, one CTA forms both M and N of a segment: twice the state warps, one production.
constexpr bool dc_both(int DP) { return DP <= 96; }
constexpr int dc_threads(int DP, int G, bool full) { return DP / 16 * ((full || !dc_both(DP) ? 1 : 2) + G) * 32; }

// RS, RP: registers of a state and of a producer thread (0: those of the launch). A warpgroup is all of one kind then, and the shares add up to
// no more than the launch's registers.
template <int DP, int G, int NS, int MINB, int RS, int RP, bool FULL>
__global__ void __launch_bounds__(dc_threads(DP, G, FULL), MINB)
delta_chunk_kernel(const VbDelta P, int nseg, float* __restrict__ ws, int* status) {
  using L = DcSmem<DP, G, NS>;
  constexpr int SW = DP / 16;                        // state warps of a matrix, and warps of a producer group
  constexpr bool BOTH = !FULL && dc_both(DP);
  constexpr int NSW = BOTH ? 2 * SW : SW;
  extern __shared__ __align__(16) uint8_t smem[];
  uint64_t *full = reinterpret_cast<uint64_t*>(smem + L::BARS), *empty = full + NS;

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mi = lane >> 3, r8 = lane & 7, g = lane >> 2, q = (lane & 3) * 2;
  const int h = blockIdx.x, seg = FULL || BOTH ? blockIdx.z : blockIdx.z >> 1, b = blockIdx.y;
  const int part = BOTH ? (warp < NSW ? warp / SW : 0) : FULL ? 0 : blockIdx.z & 1;   // 1: M
  const int d = P.d, H = P.H, W = H * d, s0 = P.cu[b], len = P.cu[b + 1] - s0;
  const int seg_len = ((len + nseg - 1) / nseg + DC_C - 1) / DC_C * DC_C;
  const int t_lo = seg * seg_len, t_hi = min(len, t_lo + seg_len);
  if (t_lo >= t_hi) return;                          // uniform over the CTA
  if (!FULL && t_hi == len) return;                  // nothing follows
  const int nch = (t_hi - t_lo + DC_C - 1) / DC_C;
  const bool values = part == 0;

  if (tid == 0) {
    for (int i = 0; i < NS; ++i) {
      mbar_init(&full[i], SW);
      mbar_init(&empty[i], NSW);
    }
    mbar_fence_init();
  }
  __syncthreads();

  const long long size = static_cast<long long>(d) * d;
  float* own = ws != nullptr ? ws + (((static_cast<long long>(b) * nseg + seg) * H + h) * 2 + part) * size : nullptr;
  bool ok = true;
  if (warp < NSW) {
    if constexpr (RS > 0) dc_more_registers<RS>();
    // ------------------------------------------------------------------ state: rows 16 warp .. of S^T
    const int e0 = warp % SW * 16;
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
    bf16* out = reinterpret_cast<bf16*>(P.out) + static_cast<long long>(s0 + t_lo + g) * P.ldo + static_cast<long long>(h) * d + e0 + q;
    // place of this lane's ldmatrix row: tokens x channels as B operand [n][k], as B operand [k][n] (transposed), v as A operand [k][m]
    // (transposed), score tiles as B operand [n][k]
    const uint32_t at_n = ((mi >> 1) * 8 + r8) * L::PITCH + (mi & 1) * 16, at_k = ((mi & 1) * 8 + r8) * L::PITCH + (mi >> 1) * 16;
    const uint32_t at_v = ((mi >> 1) * 8 + r8) * L::PITCH + (e0 + (mi & 1) * 8) * 2, at_sq = ((mi >> 1) * 8 + r8) * 48 + (mi & 1) * 16;
    int st = 0, phase = 0;
    for (int j = 0; j < nch; ++j) {
      uint8_t* stage = smem + st * L::STAGE;
      const uint32_t base = smem_u32(stage);
      if (!__all_sync(0xffffffffu, mbar_wait(&full[st], phase))) { ok = false; break; }
      // terms of a sum have accumulators of their own where registers allow: products on one accumulator wait for each other
      float Y[3][2][4] = {}, O[2][2][4] = {};
      constexpr int YM = DP <= 64 ? 2 : 1, OM = DP <= 64 ? 1 : 0;
#pragma unroll
      for (int k = 0; k < SW; ++k) {
        uint32_t sh[4], sl[4], xh[4], xl[4], xr[4];
        dc_ldsm(xh, base + L::X + at_n + k * 32);
        dc_ldsm(xl, base + L::X + L::OPER + at_n + k * 32);
        if (FULL) dc_ldsm(xr, base + L::R + at_n + k * 32);
#pragma unroll
        for (int i = 0; i < 4; ++i) dc_split(S[2 * k + (i >> 1)][(i & 1) * 2], S[2 * k + (i >> 1)][(i & 1) * 2 + 1], sh[i], sl[i]);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          dc_mma(Y[0][n], sh, xh[2 * n], xh[2 * n + 1]);
          dc_mma(Y[1][n], sh, xl[2 * n], xl[2 * n + 1]);
          if (FULL) dc_mma(O[0][n], sh, xr[2 * n], xr[2 * n + 1]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          dc_mma(Y[YM][n], sl, xh[2 * n], xh[2 * n + 1]);
          if (FULL) dc_mma(O[OM][n], sl, xr[2 * n], xr[2 * n + 1]);
        }
      }
      uint32_t v[4], zh[4], zl[4], yh[4], yl[4];
      if (values) {
        dc_ldsm_t(v, base + L::V + at_v);
        dc_ldsm(zh, base + L::Z + at_sq);
        dc_ldsm(zl, base + L::Z + DC_SQ + at_sq);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          dc_mma(Y[0][n], v, zh[2 * n], zh[2 * n + 1]);
          dc_mma(Y[1][n], v, zl[2 * n], zl[2 * n + 1]);
        }
      }
      if (FULL) {
        dc_ldsm(zh, base + L::RK + at_sq);
        dc_ldsm(zl, base + L::RB + at_sq);
#pragma unroll
        for (int n = 0; n < 2; ++n) dc_mma(O[0][n], v, zh[2 * n], zh[2 * n + 1]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int n = i >> 1, x = (i & 1) * 2;
        float y0 = Y[0][n][x] + Y[1][n][x], y1 = Y[0][n][x + 1] + Y[1][n][x + 1];
        if (YM == 2) { y0 += Y[2][n][x]; y1 += Y[2][n][x + 1]; }
        dc_split(y0, y1, yh[i], yl[i]);
      }
      if (FULL) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          dc_mma(O[0][n], yh, zl[2 * n], zl[2 * n + 1]);
          dc_mma(O[OM][n], yl, zl[2 * n], zl[2 * n + 1]);
        }
      }
      const float* wc = reinterpret_cast<const float*>(stage + L::W);
      constexpr int KB = SW < 4 ? SW : SW % 4 == 0 ? 4 : 3;   // 16-channel blocks taken together, term by term
#pragma unroll
      for (int k0 = 0; k0 < SW; k0 += KB) {
        uint32_t f[KB][4], e[KB][4];
        auto term = [&](const uint32_t (&a)[4], const uint32_t (&w)[KB][4]) {
#pragma unroll
          for (int k = 0; k < KB; ++k)
#pragma unroll
            for (int n = 0; n < 2; ++n) dc_mma(S[2 * (k0 + k) + n], a, w[k][2 * n], w[k][2 * n + 1]);
        };
#pragma unroll
        for (int k = 0; k < KB; ++k) dc_ldsm_t(f[k], base + L::B + at_k + (k0 + k) * 32);
#pragma unroll
        for (int k = 0; k < KB; ++k) dc_ldsm_t(e[k], base + L::B + L::OPER + at_k + (k0 + k) * 32);
        term(yl, f);
        term(yh, e);
        if (values) {
#pragma unroll
          for (int k = 0; k < KB; ++k) dc_ldsm_t(e[k], base + L::K + L::OPER + at_k + (k0 + k) * 32);
        }
        term(yh, f);
        if (values) {
#pragma unroll
          for (int k = 0; k < KB; ++k) dc_ldsm_t(f[k], base + L::K + at_k + (k0 + k) * 32);
          term(v, e);
          term(v, f);
        }
#pragma unroll
        for (int j2 = 2 * k0; j2 < 2 * (k0 + KB); ++j2) {
          const float2 w = *reinterpret_cast<const float2*>(wc + j2 * 8 + q);
          S[j2][0] *= w.x; S[j2][1] *= w.y; S[j2][2] *= w.x; S[j2][3] *= w.y;
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty[st]);
      if (FULL) {
        const int left = t_hi - t_lo - j * DC_C - g;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          // [e, t] -> [t, e]: this lane's token, two pairs of columns
          if (OM == 1) {
#pragma unroll
            for (int i = 0; i < 4; ++i) O[0][n][i] += O[1][n][i];
          }
          const uint32_t lo8 = dc_transpose(pack_bf16x2(O[0][n][0], O[0][n][1])), hi8 = dc_transpose(pack_bf16x2(O[0][n][2], O[0][n][3]));
          bf16* dst = out + n * 8 * P.ldo;
          if (n * 8 < left) {
            if (e0 + q < d) *reinterpret_cast<uint32_t*>(dst) = lo8;
            if (e0 + 8 + q < d) *reinterpret_cast<uint32_t*>(dst + 8) = hi8;
          }
        }
        out += DC_C * P.ldo;
      }
      if (++st == NS) { st = 0; phase ^= 1; }
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
    if constexpr (RP > 0) dc_fewer_registers<RP>();
    // ------------------------------------------------------------------ producers: group gr takes the chunks gr, gr + G, ...
    const int gr = (warp - NSW) / SW, pw = (warp - NSW) % SW, gt = pw * 32 + lane;
    uint8_t* scratch = smem + L::GROUPS + gr * L::SCRATCH;
    float *sn = reinterpret_cast<float*>(scratch + L::N), *skk = reinterpret_cast<float*>(scratch + L::KK), *siu = reinterpret_cast<float*>(scratch + L::IU);
    const uint32_t s_t = smem_u32(scratch + L::T);
    auto meet = [&]() { asm volatile("bar.sync %0, %1;" ::"r"(gr + 1), "n"(SW * 32) : "memory"); };
    // this lane's channels and tokens; token and 8 channels that this thread fetches
    const int c = pw * 16 + (lane & 7) * 2, tg = lane >> 3, ft = gt / (DP / 8), fc = gt % (DP / 8) * 8;
    const bool on = c < d;
    const bf16* prow = reinterpret_cast<const bf16*>(P.p) + static_cast<long long>(s0 + t_lo + ft) * P.ldp + h * d + fc;
    const bf16* zrow = reinterpret_cast<const bf16*>(P.zw) + static_cast<long long>(s0 + t_lo + ft) * P.ldz + h * d + fc;
    const uint32_t w0 = on ? *reinterpret_cast<const uint32_t*>(reinterpret_cast<const bf16*>(P.w0) + h * d + c) : 0u;
    const uint32_t ab = on ? *reinterpret_cast<const uint32_t*>(reinterpret_cast<const bf16*>(P.ab) + h * d + c) : 0u;
    const uint32_t f_at = smem_u32(scratch) + ft * L::PITCH + fc * 2;
    const uint8_t* raw = scratch + tg * 4 * L::PITCH + c * 2;
    auto live = [&](int j) { return fc < d && t_lo + j * DC_C + ft < t_hi ? 16u : 0u; };   // bytes to fetch; the rest is zero
    auto fetch = [&](int j) {
      const bf16 *p = prow + static_cast<long long>(j) * DC_C * P.ldp, *z = zrow + static_cast<long long>(j) * DC_C * P.ldz;
      const uint32_t n = live(j);
      if (n == 0) p = z = reinterpret_cast<const bf16*>(P.p);
      dc_fetch16(f_at, p + (n ? W : 0), n);
      dc_fetch16(f_at + L::OPER, z, n);
      dc_fetch16(f_at + 2 * L::OPER, p + (n ? 3 * W : 0), n);
      if (FULL) dc_fetch16(f_at + 3 * L::OPER, p, n);
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (gr < nch) fetch(gr);
    for (int j = gr; j < nch; j += G) {
      const int st = j % NS, n = t_hi - t_lo - j * DC_C;
      uint8_t* stage = smem + st * L::STAGE;
      const uint32_t base = smem_u32(stage);
      asm volatile("cp.async.wait_group 0;" ::: "memory");
      meet();
      uint32_t rk[4], rz[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        rk[i] = *reinterpret_cast<const uint32_t*>(raw + i * L::PITCH);
        rz[i] = *reinterpret_cast<const uint32_t*>(raw + L::OPER + i * L::PITCH);
      }
      // ---- sums of squares of the keys over the warp's channels, four tokens at once: lane pairs (l & 6) / 2 end up with a token each
      {
        float ss[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) ss[i] = dc_low(rk[i]) * dc_low(rk[i]) + dc_high(rk[i]) * dc_high(rk[i]);
        const bool up4 = (lane & 4) != 0, up2 = (lane & 2) != 0;
        const float x0 = (up4 ? ss[2] : ss[0]) + __shfl_xor_sync(0xffffffffu, up4 ? ss[0] : ss[2], 4);
        const float x1 = (up4 ? ss[3] : ss[1]) + __shfl_xor_sync(0xffffffffu, up4 ? ss[1] : ss[3], 4);
        float y = (up2 ? x1 : x0) + __shfl_xor_sync(0xffffffffu, up2 ? x0 : x1, 2);
        y += __shfl_xor_sync(0xffffffffu, y, 1);
        if ((lane & 1) == 0) skk[pw * 16 + tg * 4 + ((lane & 6) >> 1)] = y;
      }
      // ---- products of the decays: over the lane's tokens, then over the token groups
      constexpr float fall = -0.60653065971263342f * 1.4426950408889634f;      // -exp(-1/2) log2(e)
      float D0[4], D1[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const bool live = tg * 4 + i < n;
        const float x = live ? dc_ex2(fall * dc_sigmoid(dc_low(rz[i]) + dc_low(w0))) : 1.f, y = live ? dc_ex2(fall * dc_sigmoid(dc_high(rz[i]) + dc_high(w0))) : 1.f;
        D0[i] = i > 0 ? D0[i > 0 ? i - 1 : 0] * x : x;
        D1[i] = i > 0 ? D1[i > 0 ? i - 1 : 0] * y : y;
      }
      float p0 = D0[3], p1 = D1[3];
#pragma unroll
      for (int m = 8; m <= 16; m <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, p0, m), y = __shfl_up_sync(0xffffffffu, p1, m);
        if (lane >= m) { p0 *= x; p1 *= y; }
      }
      const float all0 = p0, all1 = p1;
      p0 = __shfl_up_sync(0xffffffffu, p0, 8);
      p1 = __shfl_up_sync(0xffffffffu, p1, 8);
      if (tg == 0) p0 = p1 = 1.f;                    // product in front of the lane's tokens
      // a wait that ran out is the last one: the warp goes on without, so that its group's barriers stay complete
      if (ok && j >= NS) ok = __all_sync(0xffffffffu, mbar_wait(&empty[st], ((j / NS) & 1) ^ 1));
      if (values) {
        const uint32_t m = live(j);
        dc_fetch16(base + L::V + ft * L::PITCH + fc * 2, m ? prow + static_cast<long long>(j) * DC_C * P.ldp + 2 * W : reinterpret_cast<const bf16*>(P.p), m);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
      float f0 = p0, f1 = p1;                        // W_(t-1)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        uint8_t* at = stage + (tg * 4 + i) * L::PITCH + c * 2;
        const float k0 = dc_low(rk[i]), k1 = dc_high(rk[i]);
        const uint32_t ra = *reinterpret_cast<const uint32_t*>(raw + 2 * L::OPER + i * L::PITCH), rr = *reinterpret_cast<const uint32_t*>(raw + 3 * L::OPER + i * L::PITCH);
        dc_put2(at + L::X, L::OPER, k0 * f0, k1 * f1);
        f0 = p0 * D0[i];
        f1 = p1 * D1[i];
        const float i0 = k0 * dc_rcp(f0), i1 = k1 * dc_rcp(f1);
        dc_put2(at + L::B, L::OPER, -dc_sigmoid(dc_low(ra) + dc_low(ab)) * i0, -dc_sigmoid(dc_high(ra) + dc_high(ab)) * i1);
        if (values) dc_put2(at + L::K, L::OPER, i0, i1);
        if (FULL) dc_put(at + L::R, pack_bf16x2(dc_low(rr) * f0, dc_high(rr) * f1));
      }
      if (tg == 3) *reinterpret_cast<float2*>(stage + L::W + c * 4) = make_float2(all0, all1);
      meet();
      if (j + G < nch) fetch(j + G);
      else asm volatile("cp.async.commit_group;" ::: "memory");
      // ---- scores, a matrix per warp
      const uint32_t at_m = ((mi & 1) * 8 + r8) * L::PITCH + (mi >> 1) * 16;   // A operand [m][k], and B operand [k][n] (transposed)
      const uint32_t at_n = ((mi >> 1) * 8 + r8) * L::PITCH + (mi & 1) * 16;   // B operand [n][k]
      auto product = [&](auto two, uint32_t at_a, uint32_t at_b, float (&x)[2][4]) {   // x = a b^T; two: both terms of a, else the high one
        constexpr bool TWO = decltype(two)::value;
        float m[2][2][4] = {};
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int i = 0; i < 4; ++i) x[u][i] = 0.f;
        constexpr int KB = SW < 2 ? 1 : 2;
#pragma unroll
        for (int k0 = 0; k0 < SW; k0 += KB) {
          uint32_t ah[KB][4], al[KB][4], bh[KB][4], bl[KB][4];
#pragma unroll
          for (int k = 0; k < KB; ++k) {
            dc_ldsm(ah[k], at_a + (k0 + k) * 32);
            dc_ldsm(bh[k], at_b + (k0 + k) * 32);
            dc_ldsm(bl[k], at_b + L::OPER + (k0 + k) * 32);
            if (TWO) dc_ldsm(al[k], at_a + L::OPER + (k0 + k) * 32);
          }
#pragma unroll
          for (int k = 0; k < KB; ++k)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              dc_mma(x[u], ah[k], bh[k][2 * u], bh[k][2 * u + 1]);
              dc_mma(m[0][u], ah[k], bl[k][2 * u], bl[k][2 * u + 1]);
              if (TWO) dc_mma(m[1][u], al[k], bh[k][2 * u], bh[k][2 * u + 1]);
            }
        }
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int i = 0; i < 4; ++i) x[u][i] += m[0][u][i] + (TWO ? m[1][u][i] : 0.f);
      };
#pragma unroll 1
      for (int job = pw; job < (FULL ? 4 : 2); job += SW) {                    // U B^T, U K^T, R B^T, R K^T
        if ((job & 1) && !values) continue;
        const uint32_t at_a = base + (job < 2 ? L::X : L::R) + at_m, at_b = base + ((job & 1) ? L::K : L::B) + at_n;
        float x[2][4];
        if (job < 2) product(std::true_type(), at_a, at_b, x);
        else product(std::false_type(), at_a, at_b, x);
        if (job == 1) dc_store_lower<true>(stage + L::Z, x, lane, true);
        else if (job == 2) dc_store_lower<false>(stage + L::RB, x, lane, false);
        else if (job == 3) dc_store_lower<false>(stage + L::RK, x, lane, false);
        else {
          // T = (I - tril(D U B^T D, -1))^-1 with the keys' norms D: a lane solves for a column; stored as D T D, transposed
          float kk = 1e-6f;
#pragma unroll
          for (int w = 0; w < SW; ++w) kk += skk[w * 16 + (lane & 15)];
          const float iu = rsqrtf(kk);                // of token lane % 16
          if (lane < 16) siu[lane] = iu;
          const float ig = __shfl_sync(0xffffffffu, iu, g), ig8 = __shfl_sync(0xffffffffu, iu, g + 8);
#pragma unroll
          for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
              const int s = u * 8 + q + i;
              const float is = __shfl_sync(0xffffffffu, iu, s);
              sn[s * 20 + g] = x[u][i] * ig * is;
              sn[s * 20 + g + 8] = x[u][2 + i] * ig8 * is;
            }
          __syncwarp();
          const int col = lane & 15;
          float y[DC_C];
#pragma unroll
          for (int t = 0; t < DC_C; ++t) y[t] = t == col ? 1.f : 0.f;
#pragma unroll
          for (int s = 0; s + 1 < DC_C; ++s) {        // y[s] is final: take its share from the rows below
#pragma unroll
            for (int t = (s + 1) & ~3; t < DC_C; t += 4) {
              const float4 m4 = *reinterpret_cast<const float4*>(sn + s * 20 + t);
              if (t > s) y[t] = fmaf(m4.x, y[s], y[t]);
              if (t + 1 > s) y[t + 1] = fmaf(m4.y, y[s], y[t + 1]);
              if (t + 2 > s) y[t + 2] = fmaf(m4.z, y[s], y[t + 2]);
              y[t + 3] = fmaf(m4.w, y[s], y[t + 3]);
            }
          }
#pragma unroll
          for (int t = 0; t < DC_C; t += 4) {
            const float4 f = *reinterpret_cast<const float4*>(siu + t);
            y[t] *= f.x * iu; y[t + 1] *= f.y * iu; y[t + 2] *= f.z * iu; y[t + 3] *= f.w * iu;
          }
          // lanes 0 - 15 store the high terms, the others the low ones
          uint32_t hi[8], lo[8];
#pragma unroll
          for (int t = 0; t < 8; ++t) {
            dc_split(y[2 * t], y[2 * t + 1], hi[t], lo[t]);
            if (lane >= 16) hi[t] = lo[t];
          }
          uint4* dst = reinterpret_cast<uint4*>(scratch + L::T + (lane >> 4) * DC_SQ + col * 48);
          dst[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          dst[1] = make_uint4(hi[4], hi[5], hi[6], hi[7]);
        }
      }
      meet();
      uint32_t th[4], tl[4], xh[4], xl[4];
      const uint32_t sq_m = ((mi & 1) * 8 + r8) * 48 + (mi >> 1) * 16;         // B operand [k][n] (transposed)
      const uint32_t sq_t = ((mi >> 1) * 8 + r8) * 48 + (mi & 1) * 16;         // A operand [k][m] (transposed)
      dc_ldsm_t(th, s_t + sq_t);
      dc_ldsm_t(tl, s_t + DC_SQ + sq_t);
      // ---- X = T U in U's place: the warp's channels
      {
        float x[2][4] = {}, m[2][4] = {};
        dc_ldsm_t(xh, base + L::X + at_m + pw * 32);
        dc_ldsm_t(xl, base + L::X + L::OPER + at_m + pw * 32);
#pragma unroll
        for (int u = 0; u < 2; ++u) dc_mma3(x[u], m[u], th, tl, xh[2 * u], xh[2 * u + 1], xl[2 * u], xl[2 * u + 1]);
        __syncwarp();
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int half = 0; half < 2; ++half)
            dc_put2(stage + L::X + (g + half * 8) * L::PITCH + (pw * 16 + u * 8 + q) * 2, L::OPER, x[u][half * 2] + m[u][half * 2], x[u][half * 2 + 1] + m[u][half * 2 + 1]);
      }
      // ---- Z = T tril(U K^T, -1)
      if (values && pw == 1 % SW) {
        float x[2][4] = {}, m[2][4] = {};
        dc_ldsm_t(xh, base + L::Z + sq_m);
        dc_ldsm_t(xl, base + L::Z + DC_SQ + sq_m);
#pragma unroll
        for (int u = 0; u < 2; ++u) dc_mma3(x[u], m[u], th, tl, xh[2 * u], xh[2 * u + 1], xl[2 * u], xl[2 * u + 1]);
        __syncwarp();
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int i = 0; i < 4; ++i) x[u][i] += m[u][i];
        dc_store_lower<true>(stage + L::Z, x, lane, true);
      }
      asm volatile("cp.async.wait_group 1;" ::: "memory");     // the values are there
      __syncwarp();
      if (lane == 0) mbar_arrive(&full[st]);
    }
  }
  if (!ok && lane == 0) atomicExch(status, ST_TIMEOUT_PRODUCER);
}

// Starting states of the segments: S_(g+1) = M_g S_g + N_g, in N's place. One CTA per (sequence, head, 16 columns of v); the next M is on its
// way to shared memory while one is applied.
constexpr int DF_COLS = 16, DF_RG = 256 / DF_COLS, DF_ROWS = 128 / DF_RG;
__global__ void __launch_bounds__(256)
delta_fold_kernel(const VbDelta P, int nseg, float* __restrict__ ws) {
  extern __shared__ __align__(16) float sm[];        // states [d][16], two of them; M [d][d + 4], two of them
  const int h = blockIdx.x, b = blockIdx.y, c0 = blockIdx.z * DF_COLS, d = P.d, col = threadIdx.x % DF_COLS, rg = threadIdx.x / DF_COLS;
  const int len = P.cu[b + 1] - P.cu[b], seg_len = ((len + nseg - 1) / nseg + DC_C - 1) / DC_C * DC_C, n = len > 0 ? (len + seg_len - 1) / seg_len : 0;
  const long long size = static_cast<long long>(d) * d, step = 2 * size * P.H;
  const bool c_ok = c0 + col < d, have = P.slots != nullptr && P.slots[b] >= 0 && !(P.fresh != nullptr && P.fresh[b] != 0);
  float *cur = sm, *nxt = sm + d * DF_COLS, *sM = sm + 2 * d * DF_COLS, *N = ws + (static_cast<long long>(b) * nseg * P.H + h) * 2 * size;
  const float* st = have ? P.state + static_cast<long long>(P.slots[b]) * P.slot_stride + h * size : nullptr;
  auto fetch = [&](int g) {                          // of every segment but the last
    if (g + 1 < n) {
      const uint32_t dst = smem_u32(sM + (g & 1) * d * (d + 4));
      const float* M = N + g * step + size;
      for (int i = threadIdx.x; i < d * d / 4; i += 256) dc_fetch16(dst + (i / (d / 4) * (d + 4) + i % (d / 4) * 4) * 4, M + i * 4, 16);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);
  for (int r = rg; r < d; r += DF_RG) cur[r * DF_COLS + col] = st != nullptr && c_ok ? st[static_cast<long long>(r) * d + c0 + col] : 0.f;
  for (int g = 0; g < n; ++g) {
    const bool last = g + 1 == n;
    float* at = N + g * step + c0 + col;
    float x[DF_ROWS];
#pragma unroll
    for (int i = 0; i < DF_ROWS; ++i) x[i] = !last && c_ok && i * DF_RG + rg < d ? at[static_cast<long long>(i * DF_RG + rg) * d] : 0.f;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                 // this M and the state are there, the other M's place is free
    fetch(g + 1);
    const float* m = sM + (g & 1) * d * (d + 4);
#pragma unroll
    for (int i = 0; i < DF_ROWS; ++i) {
      const int r = i * DF_RG + rg;
      if (r >= d) continue;
      if (c_ok) at[static_cast<long long>(r) * d] = cur[r * DF_COLS + col];
      if (last) continue;
#pragma unroll 4
      for (int k = 0; k < d; k += 4) {
        const float4 w = *reinterpret_cast<const float4*>(m + r * (d + 4) + k);
        x[i] = fmaf(w.x, cur[k * DF_COLS + col], x[i]);
        x[i] = fmaf(w.y, cur[(k + 1) * DF_COLS + col], x[i]);
        x[i] = fmaf(w.z, cur[(k + 2) * DF_COLS + col], x[i]);
        x[i] = fmaf(w.w, cur[(k + 3) * DF_COLS + col], x[i]);
      }
      nxt[r * DF_COLS + col] = x[i];
    }
    float* t = cur; cur = nxt; nxt = t;
  }
}

}  // namespace vb

using namespace vb;

// Segments that the prompts are cut into (1: not cut; 0: sizes that the chunked kernel does not serve).
extern "C" int vb_delta_chunk_segments(const VbDelta* p) {
  if (p->d > 128 || p->d % 8 || p->d < 8) return 0;
  const long long ctas = static_cast<long long>(p->B) * p->H;
  if (ctas <= 0) return 1;
  long long n = num_sms() * (p->d <= 64 ? 2 : 1) / ctas, most = p->T / p->B / 512;   // all segments run at once
  if (n > most) n = most;
  if (n > 32) n = 32;
  return n < 4 ? 1 : static_cast<int>(n);
}

// nseg > 1: ws holds B nseg H 2 d d floats. Returns -1 for alignments it does not serve.
extern "C" int vb_delta_chunk(const VbDelta* p, int nseg, float* ws, cudaStream_t s) {
  auto mis = [](const void* x, int n) { return (reinterpret_cast<uintptr_t>(x) & (n - 1)) != 0; };
  if (p->ldp % 8 || p->ldz % 8 || p->ldo % 2 || mis(p->p, 16) || mis(p->zw, 16) || mis(p->out, 4) || mis(p->ab, 4) || mis(p->w0, 4) || p->B > 65535 || nseg < 1 || nseg > 32) return -1;
  static int* status = nullptr;
  if (status == nullptr) cudaGetSymbolAddress(reinterpret_cast<void**>(&status), g_delta_chunk_status);
  auto go = [&](auto kern, int threads, int smem, int z) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<dim3(p->H, p->B, z), threads, smem, s>>>(*p, nseg, ws, status);
    return static_cast<int>(cudaGetLastError());
  };
#define VB_DC(DP_, G_, NS_, MINB_, RS_, RP_, FULL_) \
  go(delta_chunk_kernel<DP_, G_, NS_, MINB_, RS_, RP_, FULL_>, dc_threads(DP_, G_, FULL_), DcSmem<DP_, G_, NS_>::TOTAL, FULL_ ? nseg : (dc_both(DP_) ? 1 : 2) * (nseg - 1))
  if (nseg > 1) {
    int rc = p->d <= 32 ? VB_DC(32, 2, 4, 2, 0, 0, false) : p->d <= 64 ? VB_DC(64, 2, 4, 1, 0, 0, false) : p->d <= 96 ? VB_DC(96, 1, 4, 1, 0, 0, false) : VB_DC(128, 1, 4, 1, 0, 0, false);
    if (rc != 0) return rc;
    const int smem = (2 * p->d * DF_COLS + 2 * p->d * (p->d + 4)) * 4;
    const cudaError_t e = cudaFuncSetAttribute(delta_fold_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    delta_fold_kernel<<<dim3(p->H, p->B, (p->d + DF_COLS - 1) / DF_COLS), 256, smem, s>>>(*p, nseg, ws);
    rc = static_cast<int>(cudaGetLastError());
    if (rc != 0) return rc;
  }
  return p->d <= 32 ? VB_DC(32, 2, 4, 3, 0, 0, true) : p->d <= 64 ? VB_DC(64, 2, 4, 2, 96, 72, true) : p->d <= 96 ? VB_DC(96, 1, 4, 1, 0, 0, true) : VB_DC(128, 2, 4, 1, 112, 64, true);
#undef VB_DC
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
