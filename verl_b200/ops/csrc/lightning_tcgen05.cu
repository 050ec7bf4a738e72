// Lightning recurrence over prompts on tcgen05 tensor cores, 64 tokens at a time (bf16 q, k, v; fp32 state; query / key size <= 128).
//
// With the head's fixed decay l, inside a chunk of n tokens
//   o_t = l^(t + 1) q_t S_prev + sum_{s <= t} l^(t - s) (q_t . k_s) v_s
//   S_n = l^n S_prev + sum_s l^(n - 1 - s) k_s v_s^T
// One CTA = (sequence segment, head, 128 columns of v). Everything is transposed so that a TMEM lane is a column of v: S^T [e, d] is an
// fp32 accumulator that stays in TMEM for the whole segment, outputs are formed as O^T [e, t]. fp32 values that enter an MMA (S, the
// weighted scores, v weighted by the decay) are split into two bf16 terms, which keeps 16 mantissa bits.
//
//   warps 0 - 7    weighted values: column of v from shared memory -> two bf16 terms (A operand in TMEM), while the tensor cores are busy
//                  with the last chunk; then the state: S -> two bf16 terms (A operand in TMEM) and l^n S (accumulator), to which the
//                  update product adds. Each group of four warps takes half of the columns
//   warps 8 - 15   outputs: l^(t + 1) (S part) + (chunk part) -> bf16, lanes are consecutive columns; 32 tokens per group of four warps
//   warps 16, 17   weighted scores -> two bf16 terms in shared memory (B operand)
//   warp 18        MMA issue; warp 19: TMA (q, k, v of a chunk through a ring)
//
//   scores   [q; k] k^T      128 x 64: rows 64 .. 127 are not used (the MMA has 128 rows; k lies behind q in shared memory)
//   update   S^T += (w v)^T k      state part  S^T q^T      chunk part  v^T P^T
//
// Sequences are cut into segments when there are too few of them for the GPU: a first launch (FULL = false) computes every segment's
// own contribution to the state from nothing, a second folds them into the segments' starting states, the third is the whole.
#include "mixers.h"
#include "tcgen05_common.cuh"

#include <math.h>

namespace vb {

typedef __nv_bfloat16 bf16;
constexpr int LT_C = 64, LT_STAGES = 3, LT_THREADS = 640, LT_COLS = 128;
constexpr int LT_TILE = LT_C * 128;                     // bytes of a 64 x 64 bf16 tile
// TMEM columns
constexpr uint32_t TM_S = 0, TM_HI = 128, TM_LO = 192, TM_WHI = 256, TM_WLO = 288, TM_SC = 320, TM_OI = 384, TM_OA = 448;

template <int PD>
struct LtSmem {
  static constexpr int STAGE = (2 * PD + 2) * LT_TILE;  // per 64 query / key dimensions [q; k], then two tiles of v
  static constexpr int OFF_P = LT_STAGES * STAGE;       // weighted scores: high and low terms
  static constexpr int OFF_T = OFF_P + 2 * LT_TILE;     // tables
  static constexpr int OFF_BAR = OFF_T + (128 + 64 + 64 + 64) * 4;
  static constexpr int TOTAL = OFF_BAR + 256 + 1024;
};

__device__ int g_lightning_status[1];

// lanes x 16 columns
__device__ __forceinline__ void tmem_st_32x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(taddr), "r"(r[0]),
      "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]),
      "r"(r[14]), "r"(r[15])
      : "memory");
}
// two floats as bf16 pair plus the pair of what rounding dropped
__device__ __forceinline__ void lt_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

template <int PD, bool FULL>
__global__ void __launch_bounds__(LT_THREADS, 1)
lightning_tc_kernel(const __grid_constant__ CUtensorMap tm_qk, const __grid_constant__ CUtensorMap tm_v, const VbLightning P, int nseg, float* __restrict__ local,
                    int* status) {
  using L = LtSmem<PD>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  float* past = reinterpret_cast<float*>(smem + L::OFF_T);   // [64 + i] = l^i, zero in front
  float* up = past + 128;                                    // l^(t + 1)
  float* wfull = up + 64;                                    // l^(63 - s)
  float* wlast = wfull + 64;                                 // the same for the segment's last chunk
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);
  uint64_t *full = bars, *empty = bars + LT_STAGES;
  uint64_t *b_sc = empty + LT_STAGES, *b_p = b_sc + 1, *b_split = b_sc + 2, *b_upd = b_sc + 3, *b_int = b_sc + 4, *b_out = b_sc + 5, *b_free = b_sc + 6;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(b_sc + 7);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, quad = warp & 3;
  const int b = blockIdx.z / nseg, seg = blockIdx.z % nseg, h = blockIdx.y, c0 = blockIdx.x * LT_COLS;
  const int H = P.H, d = P.d, e = P.e;
  const int s0 = P.cu[b], len = P.cu[b + 1] - s0;
  const int seg_len = ((len + nseg - 1) / nseg + LT_C - 1) / LT_C * LT_C;
  const int t_lo = seg * seg_len, t_hi = min(len, t_lo + seg_len);
  if (t_lo >= t_hi) return;                          // uniform over the CTA, nothing allocated yet
  if (!FULL && t_hi == len) return;                  // nothing follows: the segment's own state is not needed
  const int nch = (t_hi - t_lo + LT_C - 1) / LT_C, n_last = t_hi - t_lo - (nch - 1) * LT_C;
  const float lam = P.decay[h];

  if (tid < 64) {
    past[tid] = 0.f;
    past[64 + tid] = tid == 0 ? 1.f : powf(lam, static_cast<float>(tid));
  } else if (tid < 128) {
    const int s = tid - 64;
    up[s] = powf(lam, static_cast<float>(s + 1));
    wfull[s] = s == 63 ? 1.f : powf(lam, static_cast<float>(63 - s));
    wlast[s] = s < n_last - 1 ? powf(lam, static_cast<float>(n_last - 1 - s)) : (s == n_last - 1 ? 1.f : 0.f);
  } else if (tid == 128) {
    tma_prefetch_desc(&tm_qk);
    tma_prefetch_desc(&tm_v);
    for (int i = 0; i < LT_STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(b_sc, 1);
    mbar_init(b_p, 2);
    mbar_init(b_split, 8);
    mbar_init(b_upd, 1);
    mbar_init(b_int, 1);
    mbar_init(b_out, 1);
    mbar_init(b_free, 8);
    mbar_fence_init();
  }
  if (warp == 18) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  constexpr uint32_t tmem = 0;                       // all 512 columns: the allocation starts at column 0 (checked below)
  const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
  const int row = quad * 32 + lane, ee = c0 + row;   // this lane's column of v
  const bool e_ok = ee < e;
  bool ok = *tmem_holder == tmem;
  if (!ok) {
    if (tid == 0) atomicExch(status, ST_BAD_ARGS);
  } else if (warp < 8) {
    // ------------------------------------------------------------------ weighted values and state
    const long long size = static_cast<long long>(d) * e;
    const bool have = P.slots != nullptr && P.slots[b] >= 0;
    float* slot = have ? P.state + static_cast<long long>(P.slots[b]) * P.slot_stride + h * size : nullptr;
    const float* src = nullptr;
    if (FULL) {
      if (seg > 0) src = local + ((static_cast<long long>(b) * (nseg - 1) + seg - 1) * H + h) * size;
      else if (have && P.fresh != nullptr && P.fresh[b] == 0) src = slot;
    }
    const float f_full = powf(lam, 64.f), f_last = powf(lam, static_cast<float>(n_last));
    const int group = warp >> 2, col = row & 63;
    for (int j = 0; j < nch && ok; ++j) {
      const int st = j % LT_STAGES;
      const float f = j + 1 == nch ? f_last : f_full;
      ok = mbar_wait(&full[st], (j / LT_STAGES) & 1);
      if (!ok) break;
      {
        // this group's 32 tokens of the column
        const uint8_t* v = smem + st * L::STAGE + (2 * PD + (row >> 6)) * LT_TILE + group * 32 * 128 + (col & 7) * 2;
        const float* w = (j + 1 == nch ? wlast : wfull) + group * 32;
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int i = 0; i < 16; i += 2) {
          const float4 w4 = *reinterpret_cast<const float4*>(w + 2 * i);
          float x[4];
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            const int s = 2 * i + u;
            x[u] = __uint_as_float(static_cast<uint32_t>(*reinterpret_cast<const uint16_t*>(v + s * 128 + (((col >> 3) ^ (s & 7)) << 4))) << 16);
          }
          lt_split(x[0] * w4.x, x[1] * w4.y, hi[i], lo[i]);
          lt_split(x[2] * w4.z, x[3] * w4.w, hi[i + 1], lo[i + 1]);
        }
        if (j > 0) {
          ok = mbar_wait(b_upd, (j - 1) & 1);
          tc_fence_after();
        }
        if (!ok) break;
        tmem_st_32x16(tmem + TM_WHI + group * 16 + lane_off, hi);
        tmem_st_32x16(tmem + TM_WLO + group * 16 + lane_off, lo);
      }
#pragma unroll 1
      for (int c = group * PD; c < (group + 1) * PD; ++c) {
        uint32_t x[32];
        if (j == 0) {
#pragma unroll
          for (int i = 0; i < 32; ++i) x[i] = src != nullptr && e_ok && c * 32 + i < d ? __float_as_uint(src[static_cast<long long>(c * 32 + i) * e + ee]) : 0u;
        } else {
          tmem_ld_32x32(tmem + TM_S + c * 32 + lane_off, x);
          tmem_ld_wait();
        }
        if (FULL) {
          uint32_t hi[16], lo[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) lt_split(__uint_as_float(x[2 * i]), __uint_as_float(x[2 * i + 1]), hi[i], lo[i]);
          if (c == group * PD && j > 0) {            // the terms are in use until the last state part is done
            ok = mbar_wait(b_int, (j - 1) & 1);
            tc_fence_after();
          }
          tmem_st_32x16(tmem + TM_HI + c * 16 + lane_off, hi);
          tmem_st_32x16(tmem + TM_LO + c * 16 + lane_off, lo);
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) x[i] = __float_as_uint(__uint_as_float(x[i]) * f);
        tmem_st_32x32(tmem + TM_S + c * 32 + lane_off, x);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(b_split);
    }
    if (ok) ok = mbar_wait(b_upd, (nch - 1) & 1);
    if (!ok) {
      if (lane == 0) atomicExch(status, ST_TIMEOUT_EPILOGUE);
    } else {
      tc_fence_after();
      float* dst = !FULL ? local + ((static_cast<long long>(b) * (nseg - 1) + seg) * H + h) * size : (t_hi == len ? slot : nullptr);
#pragma unroll 1
      for (int c = group * PD; c < (group + 1) * PD; ++c) {
        uint32_t x[32];
        tmem_ld_32x32(tmem + TM_S + c * 32 + lane_off, x);
        tmem_ld_wait();
        if (dst != nullptr && e_ok) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i < d) dst[static_cast<long long>(c * 32 + i) * e + ee] = __uint_as_float(x[i]);
        }
      }
    }
  } else if (warp < 16) {
    // ------------------------------------------------------------------ outputs
    if (FULL) {
      // neighbouring lanes swap, so that a lane stores two columns of every second token
      const int c = ((warp - 8) >> 2) * 32, odd = lane & 1;
      bf16* out = reinterpret_cast<bf16*>(P.out) + static_cast<long long>(s0 + t_lo + c + odd) * P.ldo + static_cast<long long>(h) * e + (ee & ~1);
      const long long step = 2 * P.ldo;
      for (int j = 0; j < nch && ok; ++j) {
        ok = mbar_wait(b_out, j & 1);
        if (!ok) break;
        tc_fence_after();
        const int n = e_ok ? (j + 1 == nch ? n_last : LT_C) - c - odd : 0;   // tokens left for this lane's rows
        bf16* dst = out + static_cast<long long>(j) * LT_C * P.ldo;
        uint32_t x[32], y[32];
        tmem_ld_32x32(tmem + TM_OI + c + lane_off, x);
        tmem_ld_32x32(tmem + TM_OA + c + lane_off, y);
        tmem_ld_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(b_free);
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float2 f = *reinterpret_cast<const float2*>(up + c + i);
          const float a0 = fmaf(f.x, __uint_as_float(x[i]), __uint_as_float(y[i])), a1 = fmaf(f.y, __uint_as_float(x[i + 1]), __uint_as_float(y[i + 1]));
          const float got = __shfl_xor_sync(0xffffffffu, odd ? a0 : a1, 1);
          if (i < n) *reinterpret_cast<uint32_t*>(dst) = odd ? pack_bf16x2(got, a1) : pack_bf16x2(a0, got);
          dst += step;
        }
      }
      if (!ok && lane == 0) atomicExch(status, ST_TIMEOUT_EPILOGUE);
    }
  } else if (warp < 18) {
    // ------------------------------------------------------------------ weighted scores: row t of [q; k] k^T
    if (FULL) {
      uint8_t* prow = smem + L::OFF_P + row * 128;
      const float* w = past + 64 + row;
      if (quad == 0) {                               // rows 0 .. 31 see no token behind 31
#pragma unroll
        for (int i = 4; i < 8; ++i) {
          const int at = (i ^ (row & 7)) << 4;
          *reinterpret_cast<uint4*>(prow + at) = make_uint4(0, 0, 0, 0);
          *reinterpret_cast<uint4*>(prow + LT_TILE + at) = make_uint4(0, 0, 0, 0);
        }
      }
      for (int j = 0; j < nch && ok; ++j) {
        ok = mbar_wait(b_sc, j & 1);
        if (!ok) break;
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c <= quad; ++c) {
          uint32_t x[32], hi[16], lo[16];
          tmem_ld_32x32(tmem + TM_SC + c * 32 + lane_off, x);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i)
            lt_split(__uint_as_float(x[2 * i]) * w[-(c * 32 + 2 * i)], __uint_as_float(x[2 * i + 1]) * w[-(c * 32 + 2 * i + 1)], hi[i], lo[i]);
          if (c == 0 && j > 0) ok = mbar_wait(b_out, (j - 1) & 1);      // the tiles are in use until the last chunk part is done
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int at = ((c * 4 + i) ^ (row & 7)) << 4;
            *reinterpret_cast<uint4*>(prow + at) = make_uint4(hi[4 * i], hi[4 * i + 1], hi[4 * i + 2], hi[4 * i + 3]);
            *reinterpret_cast<uint4*>(prow + LT_TILE + at) = make_uint4(lo[4 * i], lo[4 * i + 1], lo[4 * i + 2], lo[4 * i + 3]);
          }
        }
        fence_proxy_async_smem();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(b_p);
      }
      if (!ok && lane == 0) atomicExch(status, ST_TIMEOUT_EPILOGUE);
    }
  } else if (warp == 18) {
    // ------------------------------------------------------------------ MMA issue (the whole warp runs along: operands stay uniform)
    const bool leader = elect_one();
    constexpr uint32_t id_sc = make_idesc_f16(128, LT_C, false, false), id_upd = make_idesc_f16(128, PD * 64, false, true),
                       id_out = make_idesc_f16(128, LT_C, true, false);
    // descriptors of the first stage; other places differ in the address field (16-byte units) only
    const uint32_t s_q = smem_u32(smem), s_v = s_q + 2 * PD * LT_TILE;
    const uint64_t d_q = make_smem_desc_sw128(s_q, 16, 1024), d_k = make_smem_desc_sw128(s_q + LT_TILE, 16, 1024),
                   d_kt = make_smem_desc_sw128(s_q + LT_TILE, 2 * LT_TILE, 1024), d_vt = make_smem_desc_sw128(s_v, LT_TILE, 1024),
                   d_p = make_smem_desc_sw128(smem_u32(smem + L::OFF_P), 16, 1024);
    auto stage = [&](int j) { return static_cast<uint64_t>((j % LT_STAGES) * (L::STAGE / 16)); };
    auto wait = [&](uint64_t* bar, int parity) {
      const bool got = __all_sync(0xffffffffu, mbar_wait(bar, parity & 1));
      tc_fence_after();
      return got;
    };
    auto scores = [&](int j) {
      if (!wait(&full[j % LT_STAGES], j / LT_STAGES)) return false;
      const uint64_t a = d_q + stage(j), k_ = d_k + stage(j);
      if (leader) {
#pragma unroll
        for (int k = 0; k < PD * 4; ++k) {
          const int at = ((k >> 2) * (2 * LT_TILE) + (k & 3) * 32) / 16;
          tc_mma_f16_ss(tmem + TM_SC, a + at, k_ + at, id_sc, k > 0 ? 1u : 0u);
        }
        tc_commit(b_sc);
      }
      __syncwarp();
      return true;
    };
    if (FULL) ok = scores(0);
    for (int j = 0; j < nch && ok; ++j) {
      const uint64_t q = d_q + stage(j), kt = d_kt + stage(j), vt = d_vt + stage(j);
      if (!(ok = wait(b_split, j) && (FULL || wait(&full[j % LT_STAGES], j / LT_STAGES)))) break;
      if (leader) {
#pragma unroll
        for (int k = 0; k < 8; ++k)
          tc_mma_f16_ts(tmem + TM_S, tmem + (k >> 2 ? TM_WLO : TM_WHI) + (k & 3) * 8, kt + (k & 3) * 128, id_upd, 1u);
        tc_commit(b_upd);
      }
      __syncwarp();
      if (FULL) {
        if (j > 0 && !(ok = wait(b_free, j - 1))) break;
        if (leader) {
#pragma unroll
          for (int term = 0; term < 2; ++term)
#pragma unroll
            for (int k = 0; k < PD * 4; ++k)
              tc_mma_f16_ts(tmem + TM_OI, tmem + (term ? TM_LO : TM_HI) + k * 8, q + ((k >> 2) * (2 * LT_TILE) + (k & 3) * 32) / 16, id_sc,
                            (term > 0 || k > 0) ? 1u : 0u);
          tc_commit(b_int);
        }
        __syncwarp();
        // the scores' columns are free: those of the next chunk go ahead of this chunk's part
        if (!(ok = wait(b_p, j) && (j + 1 == nch || scores(j + 1)))) break;
        if (leader) {
#pragma unroll
          for (int k = 0; k < 8; ++k)
            tc_mma_f16_ss(tmem + TM_OA, vt + (k & 3) * 128, d_p + ((k >> 2) * LT_TILE + (k & 3) * 32) / 16, id_out, k > 0 ? 1u : 0u);
          tc_commit(b_out);
        }
        __syncwarp();
      }
      if (leader) tc_commit(&empty[j % LT_STAGES]);
      __syncwarp();
    }
    if (!ok && lane == 0) atomicExch(status, ST_TIMEOUT_MMA);
  } else {
    // ------------------------------------------------------------------ TMA
    if (lane == 0) {
      const int pv = min(2, (e - c0 + 63) / 64);
      const uint32_t bytes = static_cast<uint32_t>(((FULL ? 2 : 1) * PD + pv) * LT_TILE);
      for (int j = 0; j < nch; ++j) {
        const int st = j % LT_STAGES, t = s0 + t_lo + j * LT_C;
        if (!mbar_wait(&empty[st], ((j / LT_STAGES) & 1) ^ 1)) {
          atomicExch(status, ST_TIMEOUT_PRODUCER);
          break;
        }
        uint8_t* dst = smem + st * L::STAGE;
        mbar_expect_tx(&full[st], bytes);
#pragma unroll
        for (int c = 0; c < PD; ++c) {
          if (FULL) tma_load_3d(dst + 2 * c * LT_TILE, &tm_qk, &full[st], 64 * c, h, t);
          tma_load_3d(dst + (2 * c + 1) * LT_TILE, &tm_qk, &full[st], 64 * c, H + h, t);
        }
        for (int c = 0; c < pv; ++c) tma_load_3d(dst + (2 * PD + c) * LT_TILE, &tm_v, &full[st], c0 + 64 * c, h, t);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 18) {
    tc_fence_after();
    tmem_dealloc(*tmem_holder, 512);
  }
}

// Segment g's own state becomes the state at the start of segment g + 1 (every sequence starts from zero).
__global__ void __launch_bounds__(256)
lightning_fold_kernel(float* __restrict__ local, const float* __restrict__ decay, const int* __restrict__ cu, int nseg, int H, int size) {
  const int i = blockIdx.x * 256 + threadIdx.x, h = blockIdx.y, b = blockIdx.z;
  if (i >= size) return;
  const int len = cu[b + 1] - cu[b], seg_len = ((len + nseg - 1) / nseg + LT_C - 1) / LT_C * LT_C;
  const float f = powf(decay[h], static_cast<float>(seg_len));
  float run = 0.f;
  for (int g = 0; g + 1 < nseg && (g + 1) * seg_len < len; ++g) {
    float* at = local + ((static_cast<long long>(b) * (nseg - 1) + g) * H + h) * size + i;
    run = f * run + *at;
    *at = run;
  }
}

}  // namespace vb

using namespace vb;

// Returns -1 for sizes, strides and alignments it does not serve. nseg > 1: `local` holds B (nseg - 1) H d e floats.
extern "C" int vb_lightning_tc(const VbLightning* p, int nseg, float* local, cudaStream_t s) {
  auto mis = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) != 0; };
  if (p->d > 128 || p->d % 8 || p->e % 8 || p->d < 8 || p->e < 8 || p->ldp % 8 || mis(p->p) || p->H > 65535 || static_cast<long long>(p->B) * nseg > 65535) return -1;
  const auto bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const auto sw = CU_TENSOR_MAP_SWIZZLE_128B;
  const bf16* base = reinterpret_cast<const bf16*>(p->p);
  CUtensorMap tqk, tv;
  if (!make_tmap_3d(&tqk, base, bf, 2, p->d, 2 * p->H, p->T, p->d, p->ldp, 64, 1, LT_C, sw) ||
      !make_tmap_3d(&tv, base + 2ll * p->H * p->d, bf, 2, p->e, p->H, p->T, p->e, p->ldp, 64, 1, LT_C, sw))
    return -1;
  static int* status = nullptr;
  if (status == nullptr) cudaGetSymbolAddress(reinterpret_cast<void**>(&status), g_lightning_status);
  const dim3 grid((p->e + LT_COLS - 1) / LT_COLS, p->H, p->B * nseg);
  auto go = [&](auto kern, int smem) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<grid, LT_THREADS, smem, s>>>(tqk, tv, *p, nseg, local, status);
    return static_cast<int>(cudaGetLastError());
  };
  int rc = 0;
  if (nseg > 1) {
    rc = p->d <= 64 ? go(lightning_tc_kernel<1, false>, LtSmem<1>::TOTAL) : go(lightning_tc_kernel<2, false>, LtSmem<2>::TOTAL);
    if (rc != 0) return rc;
    const int size = p->d * p->e;
    lightning_fold_kernel<<<dim3((size + 255) / 256, p->H, p->B), 256, 0, s>>>(local, p->decay, p->cu, nseg, p->H, size);
  }
  return p->d <= 64 ? go(lightning_tc_kernel<1, true>, LtSmem<1>::TOTAL) : go(lightning_tc_kernel<2, true>, LtSmem<2>::TOTAL);
}

extern "C" int vb_lightning_status() {
  int h = 0;
  if (cudaMemcpyFromSymbol(&h, g_lightning_status, sizeof(int)) != cudaSuccess) return -1;
  if (h != 0) {
    const int z = 0;
    cudaMemcpyToSymbol(g_lightning_status, &z, sizeof(int));
  }
  return h;
}
