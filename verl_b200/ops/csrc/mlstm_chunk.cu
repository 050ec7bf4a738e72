// mLSTM over prompts, 64 tokens at a time on m16n8k16 MMAs (bf16 projections, fp32 gates and state).
//
// With b_t the cumulative log forget gate inside a chunk, a_s = i_s - b_s and M_t = max(m_prev, max_{s <= t} a_s), the
// recurrence's running maximum is m_t = b_t + M_t and
//   o_t ~ exp(m_prev - M_t) q_t S_prev + sum_{s <= t} exp(a_s - M_t) (q_t . k_s) v_s
//   S_C = exp(m_prev - M_C) S_prev + sum_s exp(a_s - M_C) k_s v_s^T
// so a chunk is three small products. One CTA = (sequence segment, head, up to 128 columns of v), the CTAs of a head form a
// cluster; a pair of warps owns 16 columns and keeps their part of S^T in fp32 accumulators for the whole segment. The accumulator layout of S^T is the B-operand layout
// of the read-out product, so S never leaves the registers; fp32 values that enter an MMA (S, the weighted scores, v weighted
// by its gate) are split into two bf16 terms, which keeps 16 mantissa bits: the per-head norm behind the read-out magnifies
// whatever is rounded where the terms of o cancel. Per-head RMS norm, weight and output gate close the chunk; the
// CTAs of a head exchange their sums of squares through distributed shared memory.
//
// Long sequences are cut into segments: a first launch (FULL = false) computes every segment's own contribution to the state
// from nothing, the second starts each segment from the fold of those before it. Compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <cooperative_groups.h>
#include <math.h>

namespace vb {

typedef __nv_bfloat16 bf16;
constexpr int MC_C = 64;          // tokens per chunk
constexpr int MC_PP = MC_C + 8;   // row pitch of the weighted score tile

struct MlstmChunkParams {
  const bf16* p; long long ldp;      // [T, q | k | v | g]
  const float* gates; long long ldg; // [T, i | f]
  const bf16 *ib, *fb;
  float cap;
  float* state; long long slot_stride;
  const int *slots, *fresh, *cu;
  float* local;                      // [B, nseg - 1, H, d e + d + 2]: segment states from nothing
  const bf16* norm;
  float eps;
  bf16* out; long long ldo;
  int H, d, e, nseg, cols;           // cols: columns of v per CTA
};

__device__ __forceinline__ uint32_t mc_smem(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void mc_cp16(void* dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mc_smem(dst)), "l"(src), "r"(ok ? 16 : 0));
}
__device__ __forceinline__ void mc_ldsm(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mc_ldsm_t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mc_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two floats as bf16 pair plus the pair of what rounding dropped
__device__ __forceinline__ void mc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 mc_unpack(uint32_t v) { return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }

constexpr int MC_THREADS = 512, MC_COLS = 128, MC_VP = MC_COLS + 8, MC_MAX_BLOCKS = 8;

template <int DP>
struct McSmem {
  static constexpr int QP = DP + 8;
  static constexpr int STAGE = (2 * MC_C * QP + MC_C * MC_VP) * 2;      // q, k, v of a chunk
  static constexpr int BUFS = DP == 256 ? 1 : 2;
  static constexpr int OFF_G = BUFS * STAGE;                            // output gates
  static constexpr int OFF_P = OFF_G + MC_C * MC_VP * 2;                // weighted scores in two bf16 terms
  static constexpr int OFF_X = OFF_P + 2 * MC_C * MC_PP * 2;            // partial read-outs exchanged by the warps of a pair
  static constexpr int OFF_F = OFF_X + 16 * 16 * 32 * 4;
  // floats: two gate buffers {a, M, dec, eneg, w [64 each], scalars [8]}, row sums [4][64], q.n [64], squares [8][64], peers [2][8][64],
  // n [DP], n parts [7][DP]
  static constexpr int GATES = 5 * MC_C + 8;
  static constexpr int FLOATS = 2 * GATES + 4 * MC_C + MC_C + 8 * MC_C + 2 * MC_MAX_BLOCKS * MC_C + 8 * DP;
  static constexpr int TOTAL = OFF_F + FLOATS * 4;
};

template <int DP, bool FULL>
__global__ void __launch_bounds__(MC_THREADS, 1)
mlstm_chunk_kernel(const MlstmChunkParams P) {
  using L = McSmem<DP>;
  namespace cg = cooperative_groups;
  constexpr int KS = DP / 16, NT = DP / 16;          // k steps of q k; 8-column tiles of S^T per warp
  constexpr int PARTS = MC_THREADS / (DP / 2) < 8 ? MC_THREADS / (DP / 2) : 8;   // token parts of the n update (two columns a thread)
  extern __shared__ __align__(16) uint8_t smem[];
  float* fl = reinterpret_cast<float*>(smem + L::OFF_F);
  float *sden = fl + 2 * L::GATES, *sqn = sden + 4 * MC_C, *sss = sqn + MC_C, *speer = sss + 8 * MC_C, *sn = speer + 2 * MC_MAX_BLOCKS * MC_C,
        *snp = sn + DP;
  bf16* sP = reinterpret_cast<bf16*>(smem + L::OFF_P);
  bf16* sG = reinterpret_cast<bf16*>(smem + L::OFF_G);
  float* sX = reinterpret_cast<float*>(smem + L::OFF_X);
  // two warps share 16 columns of v (wg): each holds half of the d columns of S^T and finishes half of the tokens (hw)
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wg = warp & 7, hw = warp >> 3;
  const int b = blockIdx.z / P.nseg, seg = blockIdx.z % P.nseg, h = blockIdx.y, c0 = blockIdx.x * P.cols;
  const int H = P.H, d = P.d, e = P.e;
  const int s0 = P.cu[b], len = P.cu[b + 1] - s0;
  const int seg_len = ((len + P.nseg - 1) / P.nseg + MC_C - 1) / MC_C * MC_C;
  const int t_lo = seg * seg_len, t_hi = min(len, t_lo + seg_len);
  if (t_lo >= t_hi) return;                          // the same for every CTA of a cluster
  if (!FULL && t_hi == len) return;                  // nothing follows: the segment's own state is not needed
  const int e0 = c0 + wg * 16, d0 = hw * (DP / 2);   // first column and first d of this warp
  const bool e_ok = e0 < e && wg * 16 < P.cols;
  const int er = lane >> 2, kc = (lane & 3) * 2, mi = lane >> 3, r8 = lane & 7;
  const long long lsize = static_cast<long long>(d) * e + d + 2;
  const bool have = P.slots != nullptr && P.slots[b] >= 0;
  float* slot = have ? P.state + static_cast<long long>(P.slots[b]) * P.slot_stride : nullptr;
  float* slot_S = have ? slot + static_cast<long long>(h) * d * e : nullptr;
  float* slot_n = have ? slot + static_cast<long long>(H) * d * e + h * d : nullptr;
  float* slot_m = have ? slot + static_cast<long long>(H) * d * e + H * d + h : nullptr;

  // ---- S^T accumulators: tile j covers d columns [d0 + 8j, + 8); element (e0 + er (+ 8), d0 + 8j + kc (+ 1))
  float S[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.f;
  auto each = [&](auto fn) {                         // fn(element, d row, e column) over this thread's valid elements
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int dd = d0 + j * 8 + kc + (i & 1), ee = e0 + er + (i >> 1) * 8;
        if (e_ok && dd < d && ee < e) fn(S[j][i], dd, ee);
      }
  };
  float m_prev = FULL ? 0.f : -INFINITY, f_total = 0.f;
  for (int r = tid; r < DP; r += MC_THREADS) sn[r] = 0.f;
  for (int r = tid; r < 7 * DP; r += MC_THREADS) snp[r] = 0.f;
  if (FULL) {
    if (have && P.fresh != nullptr && P.fresh[b] == 0) {
      each([&](float& v, int dd, int ee) { v = slot_S[static_cast<long long>(dd) * e + ee]; });
      for (int r = tid; r < d; r += MC_THREADS) sn[r] = slot_n[r];
      m_prev = *slot_m;
    }
    for (int g = 0; g < seg; ++g) {                  // fold of the segments before this one
      const float* loc = P.local + ((static_cast<long long>(b) * (P.nseg - 1) + g) * H + h) * lsize;
      const float m_loc = loc[lsize - 2], F = loc[lsize - 1];
      const float m = fmaxf(F + m_prev, m_loc), keep = expf(F + m_prev - m), add = expf(m_loc - m);
      each([&](float& v, int dd, int ee) { v = keep * v + add * loc[static_cast<long long>(dd) * e + ee]; });
      for (int r = tid; r < d; r += MC_THREADS) sn[r] = keep * sn[r] + add * loc[static_cast<long long>(d) * e + r];
      m_prev = m;
    }
  }
  float wn[2][2] = {};                               // norm weights of this thread's columns
  if (FULL && e_ok)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int u = 0; u < 2; ++u)
        if (e0 + n * 8 + kc + u < e) wn[n][u] = to_f(P.norm[h * e + e0 + n * 8 + kc + u]);

  const bf16* base = P.p + static_cast<long long>(s0) * P.ldp;
  const int vw = min(P.cols, e - c0) / 8;            // 16-byte pieces of a v or g row
  auto load_v = [&](bf16* dst, int t0, long long off) {
    for (int i = tid; i < MC_C * (MC_COLS / 8); i += MC_THREADS) {
      const int r = i / (MC_COLS / 8), c = i % (MC_COLS / 8);
      const bool ok = t0 + r < t_hi && c < vw;
      mc_cp16(dst + r * MC_VP + c * 8, ok ? base + static_cast<long long>(t0 + r) * P.ldp + off + c * 8 : base, ok);
    }
  };
  auto load = [&](int st, int t0) {
    bf16* q = reinterpret_cast<bf16*>(smem + st * L::STAGE);
    bf16* k = q + MC_C * L::QP;
    for (int i = tid; i < MC_C * (DP / 8); i += MC_THREADS) {
      const int r = i / (DP / 8), c = (i % (DP / 8)) * 8;
      const bool ok = t0 + r < t_hi && c < d;
      const bf16* row = base + static_cast<long long>(t0 + r) * P.ldp;
      if (FULL) mc_cp16(q + r * L::QP + c, ok ? row + h * d + c : base, ok);
      mc_cp16(k + r * L::QP + c, ok ? row + (H + h) * d + c : base, ok);
    }
    load_v(k + MC_C * L::QP, t0, 2 * H * d + static_cast<long long>(h) * e + c0);
    asm volatile("cp.async.commit_group;");
  };
  const float ibv = to_f(P.ib[h]), fbv = to_f(P.fb[h]);
  const float qs = 1.f / sqrtf(static_cast<float>(d)), inv_e = 1.f / e;
  float gi[2], gf[2];                                // gate pre-activations of the next chunk (warp 0, two tokens per lane)
  auto fetch_gates = [&](int t0) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = t0 + lane * 2 + u;
      const float* g = P.gates + static_cast<long long>(s0 + t) * P.ldg;
      gi[u] = t < t_hi ? g[h] : 0.f;
      gf[u] = t < t_hi ? g[H + h] : 0.f;
    }
  };
  // Gates of the chunk at t0 into buffer `buf` (one warp; its score block lies above the diagonal, so it has the time), and the
  // request for those of the chunk after it.
  float m_run = m_prev;
  auto gates = [&](int t0, int buf) {
    float *sa = fl + buf * L::GATES, *sM = sa + MC_C, *sdec = sM + MC_C, *sneg = sdec + MC_C, *sw = sneg + MC_C, *sc = sw + MC_C;
    float il[2], ff[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const bool ok = t0 + lane * 2 + u < t_hi;
      il[u] = ok ? P.cap * tanhf((gi[u] + ibv) / P.cap) : -INFINITY;
      ff[u] = ok ? log_sigmoid(P.cap * tanhf((gf[u] + fbv) / P.cap)) : 0.f;
    }
    fetch_gates(t0 + MC_C);
    float run = ff[0] + ff[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += x;
    }
    const float b1 = run, b0 = run - ff[1];
    const float a0 = il[0] - b0, a1 = il[1] - b1;
    float mx = fmaxf(a0, a1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, mx, o);
      if (lane >= o) mx = fmaxf(mx, x);
    }
    float before = __shfl_up_sync(0xffffffffu, mx, 1);
    if (lane == 0) before = -INFINITY;
    const float M0 = fmaxf(m_run, fmaxf(before, a0)), M1 = fmaxf(m_run, mx);
    const float MC = __shfl_sync(0xffffffffu, M1, 31), bC = __shfl_sync(0xffffffffu, b1, 31);
    const float aa[2] = {a0, a1}, MM[2] = {M0, M1}, bb[2] = {b0, b1};
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = lane * 2 + u;
      sa[t] = aa[u];
      sM[t] = MM[u];
      sdec[t] = expf(m_run - MM[u]);
      sneg[t] = expf(-(bb[u] + MM[u]));
      sw[t] = expf(aa[u] - MC);
    }
    if (lane == 0) {
      sc[0] = expf(m_run - MC);
      sc[1] = bC + MC;
      sc[2] = bC;
    }
    m_run = bC + MC;
  };
  load(0, t_lo);
  if (warp == 1) {
    fetch_gates(t_lo);
    gates(t_lo, 0);
  }
  cg::cluster_group cluster = cg::this_cluster();
  const int nblk = gridDim.x;
  if (nblk > 1) cluster.sync();                      // peers run, and have read the stored state, before anything is replaced
  __syncthreads();
  int st = 0;
  for (int t0 = t_lo; t0 < t_hi; t0 += MC_C, st ^= L::BUFS - 1) {
    for (int r = tid; r < DP; r += MC_THREADS) {      // the parts of the last chunk's n update
#pragma unroll
      for (int u = 0; u < PARTS - 1; ++u) sn[r] += snp[u * DP + r];
    }
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();                                  // A: chunk and gates are in shared memory, the other stage is free
    const bool more = t0 + MC_C < t_hi;
    if (FULL) {
      load_v(sG, t0, 2 * H * d + static_cast<long long>(H + h) * e + c0);
      asm volatile("cp.async.commit_group;");
    }
    if (L::BUFS == 2 && more) load(st ^ 1, t0 + MC_C);
    const bf16* q = reinterpret_cast<const bf16*>(smem + st * L::STAGE);
    const bf16* k = q + MC_C * L::QP;
    const uint32_t uq = mc_smem(q), uk = mc_smem(k), uv = mc_smem(k + MC_C * L::QP), uP = mc_smem(sP);
    const int par = ((t0 - t_lo) / MC_C) & 1;
    const float *sa = fl + par * L::GATES, *sM = sa + MC_C, *sdec = sM + MC_C, *sneg = sdec + MC_C, *sw = sneg + MC_C, *sc = sw + MC_C;
    const float decC = sc[0], m_next = sc[1];
    if (warp == 1 && more) gates(t0 + MC_C, par ^ 1);
    float o[2][2][4] = {};
    if (FULL) {
      // ---- weighted scores P = exp(a_s - M_t) q_t . k_s: a warp owns a 16 x 16 block, zero above the diagonal
      {
        const int tb = (warp >> 2) * 16, sb = (warp & 3) * 16;
        float acc[2][4] = {};
        if (sb <= tb) {
#pragma unroll
          for (int kk = 0; kk < KS; ++kk) {
            uint32_t fa[4], fb[4];
            mc_ldsm(fa, uq + ((tb + (mi & 1) * 8 + r8) * L::QP + kk * 16 + (mi >> 1) * 8) * 2);
            mc_ldsm(fb, uk + ((sb + (mi >> 1) * 8 + r8) * L::QP + kk * 16 + (mi & 1) * 8) * 2);
            mc_mma(acc[0], fa, fb[0], fb[1]);
            mc_mma(acc[1], fa, fb[2], fb[3]);
          }
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int t = tb + er + half * 8;
          const float Mt = sM[t];
          float rs = 0.f;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            float x[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              const int s = sb + j * 8 + kc + u;
              x[u] = s <= t ? acc[j][half * 2 + u] * qs * __expf(sa[s] - Mt) : 0.f;
              rs += x[u];
            }
            uint32_t hi, lo;
            mc_split(x[0], x[1], hi, lo);
            *reinterpret_cast<uint32_t*>(sP + t * MC_PP + sb + j * 8 + kc) = hi;
            *reinterpret_cast<uint32_t*>(sP + (MC_C + t) * MC_PP + sb + j * 8 + kc) = lo;
          }
          rs += __shfl_xor_sync(0xffffffffu, rs, 1);
          rs += __shfl_xor_sync(0xffffffffu, rs, 2);
          if ((lane & 3) == 0) sden[(warp & 3) * MC_C + t] = rs;
        }
      }
      // ---- q_t . n_prev: eight lanes per token
      {
        const int t = tid >> 3;
        float x = 0.f;
#pragma unroll 4
        for (int c = (tid & 7) * 2; c < DP; c += 16) {
          const float2 qq = mc_unpack(*reinterpret_cast<const uint32_t*>(q + t * L::QP + c));
          x += qq.x * sn[c] + qq.y * sn[c + 1];
        }
        x += __shfl_xor_sync(0xffffffffu, x, 1);
        x += __shfl_xor_sync(0xffffffffu, x, 2);
        x += __shfl_xor_sync(0xffffffffu, x, 4);
        if ((tid & 7) == 0) sqn[t] = x * qs;
      }
      // ---- read-out of this warp's half of the state for all tokens; the pair swaps the halves it does not finish
      {
        float r[4][2][4] = {};
        if (e_ok) {
          uint32_t fa[2][4];                          // query fragments, one product ahead
          auto fetch = [&](int i) {
            mc_ldsm(fa[i & 1], uq + (((i & 3) * 16 + (mi & 1) * 8 + r8) * L::QP + d0 + (i >> 2) * 16 + (mi >> 1) * 8) * 2);
          };
          fetch(0);
#pragma unroll
          for (int kk = 0; kk < KS / 2; ++kk) {
            uint32_t h0, l0, h1, l1, h2, l2, h3, l3;
            mc_split(S[2 * kk][0], S[2 * kk][1], h0, l0);
            mc_split(S[2 * kk + 1][0], S[2 * kk + 1][1], h1, l1);
            mc_split(S[2 * kk][2], S[2 * kk][3], h2, l2);
            mc_split(S[2 * kk + 1][2], S[2 * kk + 1][3], h3, l3);
#pragma unroll
            for (int m = 0; m < 4; ++m) {
              if (kk * 4 + m + 1 < KS * 2) fetch(kk * 4 + m + 1);
              mc_mma(r[m][0], fa[m & 1], h0, h1);
              mc_mma(r[m][1], fa[m & 1], h2, h3);
              mc_mma(r[m][0], fa[m & 1], l0, l1);
              mc_mma(r[m][1], fa[m & 1], l2, l3);
            }
          }
        }
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              sX[((warp * 2 + m) * 8 + n * 4 + i) * 32 + lane] = hw ? r[m][n][i] : r[2 + m][n][i];
              o[m][n][i] = hw ? r[2 + m][n][i] : r[m][n][i];
            }
      }
      __syncthreads();                                // B: scores, row sums, partial read-outs
      if (e_ok) {
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i)
              o[m][n][i] = (o[m][n][i] + sX[(((warp ^ 8) * 2 + m) * 8 + n * 4 + i) * 32 + lane]) * (sdec[hw * 32 + m * 16 + (i >> 1) * 8 + er] * qs);
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {              // the chunk's own tokens
          if (kk >= 2 + 2 * hw) continue;
          uint32_t fv[4];
          mc_ldsm_t(fv, uv + ((kk * 16 + (mi & 1) * 8 + r8) * MC_VP + wg * 16 + (mi >> 1) * 8) * 2);
#pragma unroll
          for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int term = 0; term < 2; ++term) {
              uint32_t fa[4];
              mc_ldsm(fa, uP + ((term * MC_C + hw * 32 + m * 16 + (mi & 1) * 8 + r8) * MC_PP + kk * 16 + (mi >> 1) * 8) * 2);
              mc_mma(o[m][0], fa, fv[0], fv[1]);
              mc_mma(o[m][1], fa, fv[2], fv[3]);
            }
        }
      }
      // ---- denominator; sum of squares over the head
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int t = hw * 32 + m * 16 + half * 8 + er;
          const float den = sdec[t] * sqn[t] + ((sden[t] + sden[MC_C + t]) + (sden[2 * MC_C + t] + sden[3 * MC_C + t]));
          const float inv = __fdividef(1.f, fmaxf(fabsf(den), sneg[t]) + 1e-6f);
          float ss = 0.f;
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              float& x = o[m][n][half * 2 + u];
              x *= inv;
              ss += x * x;
            }
          ss += __shfl_xor_sync(0xffffffffu, ss, 1);
          ss += __shfl_xor_sync(0xffffffffu, ss, 2);
          if ((lane & 3) == 0) sss[wg * MC_C + t] = ss;
        }
      if (L::BUFS == 2 && more) asm volatile("cp.async.wait_group 1;");
      else asm volatile("cp.async.wait_group 0;");
      __syncthreads();                                // C: sums of squares, output gates
      if (nblk > 1) {
        if (tid < MC_C) {
          float ss = 0.f;
#pragma unroll
          for (int w = 0; w < 8; ++w) ss += sss[w * MC_C + tid];
          for (int r = 0; r < nblk; ++r) cluster.map_shared_rank(speer, r)[(par * MC_MAX_BLOCKS + blockIdx.x) * MC_C + tid] = ss;
        }
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
      }
    }
    // ---- state update: S^T = decC S^T + (w v)^T k
    if (e_ok) {
#pragma unroll
      for (int j = 0; j < NT; ++j) { S[j][0] *= decC; S[j][1] *= decC; S[j][2] *= decC; S[j][3] *= decC; }
#pragma unroll
      for (int kk = 0; kk < MC_C / 16; ++kk) {
        uint32_t fv[4], hi[4], lo[4];
        // (w v)^T as A: rows = v columns, k = tokens; registers {e0 s0, e8 s0, e0 s8, e8 s8}
        mc_ldsm_t(fv, uv + ((kk * 16 + (mi >> 1) * 8 + r8) * MC_VP + wg * 16 + (mi & 1) * 8) * 2);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int s = kk * 16 + (i >> 1) * 8 + kc;
          const float2 x = mc_unpack(fv[i]);
          mc_split(x.x * sw[s], x.y * sw[s + 1], hi[i], lo[i]);
        }
        uint32_t fk[2][4];                            // key fragments, one product ahead
        auto fetch = [&](int j) { mc_ldsm_t(fk[j & 1], uk + ((kk * 16 + (mi & 1) * 8 + r8) * L::QP + d0 + j * 16 + (mi >> 1) * 8) * 2); };
        fetch(0);
#pragma unroll
        for (int j = 0; j < NT / 2; ++j) {
          if (j + 1 < NT / 2) fetch(j + 1);
          mc_mma(S[2 * j], hi, fk[j & 1][0], fk[j & 1][1]);
          mc_mma(S[2 * j + 1], hi, fk[j & 1][2], fk[j & 1][3]);
          mc_mma(S[2 * j], lo, fk[j & 1][0], fk[j & 1][1]);
          mc_mma(S[2 * j + 1], lo, fk[j & 1][2], fk[j & 1][3]);
        }
      }
    }
    if (tid < DP / 2 * PARTS) {
      const int r = tid % (DP / 2) * 2, part = tid / (DP / 2);
      float x0 = part == 0 ? decC * sn[r] : 0.f, x1 = part == 0 ? decC * sn[r + 1] : 0.f;
#pragma unroll
      for (int s = part * (MC_C / PARTS); s < (part + 1) * (MC_C / PARTS); s += 4) {
        const float4 w = *reinterpret_cast<const float4*>(sw + s);
        const float ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float2 kk = mc_unpack(*reinterpret_cast<const uint32_t*>(k + (s + u) * L::QP + r));
          x0 += ww[u] * kk.x;
          x1 += ww[u] * kk.y;
        }
      }
      float* dst = part == 0 ? sn + r : snp + (part - 1) * DP + r;
      dst[0] = x0;
      dst[1] = x1;
    }
    if (FULL) {
      // ---- norm over the head, weight, output gate
      if (nblk > 1) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
      if (e_ok) {
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int t = hw * 32 + m * 16 + half * 8 + er;
            float ss = 0.f;
            if (nblk > 1) {
              for (int r = 0; r < nblk; ++r) ss += speer[(par * MC_MAX_BLOCKS + r) * MC_C + t];
            } else {
#pragma unroll
              for (int w = 0; w < 8; ++w) ss += sss[w * MC_C + t];
            }
            const float rs = rsqrtf(ss * inv_e + P.eps);
            bf16* dst = P.out + static_cast<long long>(s0 + t0 + t) * P.ldo + h * e + e0 + kc;
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              const float2 g = mc_unpack(*reinterpret_cast<const uint32_t*>(sG + t * MC_VP + wg * 16 + n * 8 + kc));
              const float y0 = __fdividef(o[m][n][half * 2] * rs * wn[n][0], 1.f + __expf(-g.x));
              const float y1 = __fdividef(o[m][n][half * 2 + 1] * rs * wn[n][1], 1.f + __expf(-g.y));
              if (t0 + t < t_hi && e0 + n * 8 + kc < e) *reinterpret_cast<__nv_bfloat162*>(dst + n * 8) = __floats2bfloat162_rn(y0, y1);
            }
          }
      }
    }
    m_prev = m_next;
    f_total += sc[2];
    __syncthreads();                                  // D: gates, n and the chunk may be replaced
    if (L::BUFS == 1 && more) load(0, t0 + MC_C);
  }
  for (int r = tid; r < DP; r += MC_THREADS)
#pragma unroll
    for (int u = 0; u < PARTS - 1; ++u) sn[r] += snp[u * DP + r];
  // ---- final state of the sequence, or this segment's own state
  if (!FULL) {
    float* loc = P.local + ((static_cast<long long>(b) * (P.nseg - 1) + seg) * H + h) * lsize;
    each([&](float& v, int dd, int ee) { loc[static_cast<long long>(dd) * e + ee] = v; });
    if (blockIdx.x == 0) {
      for (int r = tid; r < d; r += MC_THREADS) loc[static_cast<long long>(d) * e + r] = sn[r];
      if (tid == 0) { loc[lsize - 2] = m_prev; loc[lsize - 1] = f_total; }
    }
  } else if (have && t_hi == len) {
    each([&](float& v, int dd, int ee) { slot_S[static_cast<long long>(dd) * e + ee] = v; });
    if (blockIdx.x == 0) {
      for (int r = tid; r < d; r += MC_THREADS) slot_n[r] = sn[r];
      if (tid == 0) *slot_m = m_prev;
    }
  }
}

static int mc_dp(int d) { return d <= 64 ? 64 : (d <= 128 ? 128 : 256); }

template <int DP>
static int mc_launch(const MlstmChunkParams& p, int B, int blocks, cudaStream_t s) {
  auto go = [&](auto kern) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, McSmem<DP>::TOTAL);
    if (e != cudaSuccess) return static_cast<int>(e);
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(blocks, p.H, B * p.nseg);
    cfg.blockDim = dim3(MC_THREADS);
    cfg.dynamicSmemBytes = McSmem<DP>::TOTAL;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = blocks;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return static_cast<int>(cudaLaunchKernelEx(&cfg, kern, p));
  };
  int rc = p.nseg > 1 ? go(mlstm_chunk_kernel<DP, false>) : 0;
  if (rc == 0) rc = go(mlstm_chunk_kernel<DP, true>);
  return rc;
}

}  // namespace vb

using namespace vb;

// Segments a sequence is cut into (1 = none; the workspace then needs B * (nseg - 1) * H * (d e + d + 2) floats), or 0 when the
// sizes are not served. all_fresh: every sequence starts from zero.
extern "C" int vb_mlstm_chunk_segments(int T, int B, int H, int d, int e, int all_fresh) {
  const int blocks = (e + MC_COLS - 1) / MC_COLS;
  if (d % 8 || e % 8 || d > 256 || d < 8 || e < 8 || blocks > MC_MAX_BLOCKS || B > 65535 || H > 65535) return 0;
  if (!all_fresh) return 1;
  int s = 148 / (B * H * blocks);
  const int by_len = T / B / (4 * MC_C);
  if (s > by_len) s = by_len;
  if (s > 32) s = 32;
  return (s < 1 || static_cast<long long>(B) * s > 65535) ? 1 : s;
}

extern "C" int vb_mlstm_chunk(const void* qkvg, long long ldp, const float* gates, long long ldg, const void* ib, const void* fb, float cap,
                              float* state, long long slot_stride, const int* slots, const int* fresh, const int* cu, int B, int nseg, float* local,
                              const void* norm, float eps, void* out, long long ldo, int H, int d, int e, cudaStream_t s) {
  if (ldp % 8 || (reinterpret_cast<uintptr_t>(qkvg) & 15) || (ldo % 2) || (reinterpret_cast<uintptr_t>(out) & 3)) return -1;
  MlstmChunkParams p{};
  p.p = reinterpret_cast<const bf16*>(qkvg); p.ldp = ldp; p.gates = gates; p.ldg = ldg;
  p.ib = reinterpret_cast<const bf16*>(ib); p.fb = reinterpret_cast<const bf16*>(fb); p.cap = cap;
  p.state = state; p.slot_stride = slot_stride; p.slots = slots; p.fresh = fresh; p.cu = cu; p.local = local;
  p.norm = reinterpret_cast<const bf16*>(norm); p.eps = eps; p.out = reinterpret_cast<bf16*>(out); p.ldo = ldo;
  p.H = H; p.d = d; p.e = e; p.nseg = nseg;
  int blocks = (e + MC_COLS - 1) / MC_COLS;
  p.cols = ((e + blocks - 1) / blocks + 15) / 16 * 16;
  blocks = (e + p.cols - 1) / p.cols;
  switch (mc_dp(d)) {
    case 64: return mc_launch<64>(p, B, blocks, s);
    case 128: return mc_launch<128>(p, B, blocks, s);
    default: return mc_launch<256>(p, B, blocks, s);
  }
}
