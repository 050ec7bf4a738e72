// Prompt attention of the mixer stacks on tcgen05 tensor cores: causal, windowed (with kept first keys) or chunked, with a sink, capped scores
// and an output gate.
// Latent attention, or grouped-query attention with query / key and value sizes of its own (no rotated part, kv_group query
// heads per key head).
//
// One CTA = (sequence, NT query tiles of 128 rows, head): one tile where two such CTAs fit an SM (the softmax, start and end of
// one run under the products of the other), else two tiles that share the key blocks, else one. The score product runs over two operand groups, the head's
// unrotated key part and the rotated part shared by all heads, accumulated in the same TMEM tile, so keys are never
// concatenated in memory. Only key blocks that some row of a tile can see are loaded and multiplied.
//
//   warp 0        TMA: query tiles once, then key and value blocks of 64 through two 2-stage rings (a key stage is free as soon
//                 as its scores are done, a value stage after its product)
//   warp 1        MMA: S_t(j + 1) is issued ahead of O_t += P_t(j) V(j); the tiles alternate, so one tile's softmax runs under
//                 the other's products
//   warps 2 + 4t  softmax of tile t: thread == query row; the running maximum starts at the sink (weight 1, no value); O is
//   .. 5 + 4t     rescaled only when a row's maximum grew by more than 2^8
// Epilogue: O / l * sigmoid(gate) -> bf16 [T, H, dv].
// Differential attention (PAIR): the two tiles are the two maps of the same 128 query rows; their key blocks stand behind each other in
// a stage, the value blocks are shared. The epilogue forms the difference of the maps and norms it: a row's columns are divided
// between its two threads (one per map), which exchange denominators and sums of squares through shared memory.
#include "mixers.h"
#include "tcgen05_common.cuh"

#include <math.h>

namespace vb {

constexpr int LP_BQ = 128, LP_BK = 64;

struct LatentPrefillParams {
  const int* cu_q;
  const int* cu_k;
  int num_seqs, dv, window, keep, chunk, kv_group, pu, pr, pv, su, sr;  // panels of 64 columns (unrotated, rotated, value), k steps of 16
  const __nv_bfloat16* sink;
  const float* gate;
  long long ldg;
  __nv_bfloat16* out;
  long long ldo;
  float scale_log2;
  // CAP: score = cap_log2 * tanh(x * cap_z) of the product x, in powers of two. Where |x| <= cap_near: x times a polynomial in
  // x^2 with coefficients cap_poly
  float cap_z, cap_log2, cap_near, cap_poly[5];
  int tmem_cols;
  int* status;
  const __nv_bfloat16* diff_vec;   // PAIR: four vectors of du entries
  int du, key_maps;                // key_maps 2: key heads are maps, two per value head
  float diff, eps;
};

__device__ int g_latent_prefill_status[1];

// two fp32 values in a 64-bit register pair: one instruction for both
__device__ __forceinline__ uint64_t pack2(uint32_t a, uint32_t b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "r"(a), "r"(b));
  return r;
}
__device__ __forceinline__ uint64_t both2(float v) { return pack2(__float_as_uint(v), __float_as_uint(v)); }
__device__ __forceinline__ void unpack2(uint64_t v, uint32_t& a, uint32_t& b) { asm("mov.b64 {%0, %1}, %2;" : "=r"(a), "=r"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.ftz.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.ftz.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.ftz.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

// Columns of a row of both maps' products -> (1 - diff) rms_norm(a0 - lambda a1). Threads (t = 0, 1; r) share row r: they take every
// second group of 32 columns. The query tiles' place in shared memory, long read, holds what they exchange.
__device__ __forceinline__ void pair_epilogue(const LatentPrefillParams& p, uint8_t* smem, uint32_t o_base, int t, int r, int lane, float inv_l, bool row_ok,
                                              long long tok, int head) {
  float *s_inv = reinterpret_cast<float*>(smem), *s_sum = s_inv + 2 * LP_BQ;
  float x = 0.f, y = 0.f;
  for (int i = lane; i < p.du; i += 32) {
    x = fmaf(__bfloat162float(p.diff_vec[i]), __bfloat162float(p.diff_vec[p.du + i]), x);
    y = fmaf(__bfloat162float(p.diff_vec[2 * p.du + i]), __bfloat162float(p.diff_vec[3 * p.du + i]), y);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    x += __shfl_xor_sync(0xffffffffu, x, o);
    y += __shfl_xor_sync(0xffffffffu, y, o);
  }
  const float lam = expf(x) - expf(y) + p.diff;
  s_inv[t * LP_BQ + r] = inv_l;
  tc_fence_before();
  asm volatile("bar.sync 1, 256;" ::: "memory");   // the softmax warps of both maps: both products are complete
  tc_fence_after();
  const float f0 = s_inv[r], f1 = -lam * s_inv[LP_BQ + r];
  float ss = 0.f;
  for (int c = t; c < p.pv * 2; c += 2) {
    uint32_t a[32], b[32];
    tmem_ld_32x32(o_base + c * 32, a);
    tmem_ld_32x32(o_base + p.pv * 64 + c * 32, b);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      const float z = fmaf(__uint_as_float(a[i]), f0, __uint_as_float(b[i]) * f1);
      ss = fmaf(z, z, ss);                          // columns past dv are zero
    }
  }
  s_sum[t * LP_BQ + r] = ss;
  asm volatile("bar.sync 1, 256;" ::: "memory");
  const float g = (1.f - p.diff) * rsqrtf((s_sum[r] + s_sum[LP_BQ + r]) / p.dv + p.eps);
  for (int c = t; c < p.pv * 2; c += 2) {
    uint32_t a[32], b[32];
    tmem_ld_32x32(o_base + c * 32, a);
    tmem_ld_32x32(o_base + p.pv * 64 + c * 32, b);
    tmem_ld_wait();
    if (!row_ok) continue;
    __nv_bfloat16* dst = p.out + tok * p.ldo + static_cast<long long>(head) * p.dv + c * 32;
#pragma unroll
    for (int i = 0; i < 32; i += 8) {
      if (c * 32 + i < p.dv) {
        uint32_t v[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int j = i + 2 * k;
          v[k] = pack_bf16x2(g * fmaf(__uint_as_float(a[j]), f0, __uint_as_float(b[j]) * f1), g * fmaf(__uint_as_float(a[j + 1]), f0, __uint_as_float(b[j + 1]) * f1));
        }
        *reinterpret_cast<uint4*>(dst + i) = make_uint4(v[0], v[1], v[2], v[3]);
      }
    }
  }
}

template <int NT, bool CAP, bool PAIR>
__global__ void __launch_bounds__(64 + 128 * NT, 3 - NT)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tm_qu, const __grid_constant__ CUtensorMap tm_qr, const __grid_constant__ CUtensorMap tm_ku,
                      const __grid_constant__ CUtensorMap tm_kr, const __grid_constant__ CUtensorMap tm_v, const LatentPrefillParams p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = smem_raw;
  if ((smem_u32(smem) & 1023u) != 0u) {  // the swizzled layouts need 1024-byte aligned tiles; there is no slack for rounding up
    if (threadIdx.x == 0) atomicExch(p.status, 9);
    return;
  }
  constexpr int RT = PAIR ? 1 : NT;   // row tiles
  const int qp = p.pu + p.pr;
  const int q_bytes = qp * (LP_BQ * 128), map_bytes = qp * (LP_BK * 128), k_bytes = (PAIR ? 2 : 1) * map_bytes, v_bytes = p.pv * (LP_BK * 128);
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + NT * q_bytes;
  uint8_t* sV = sK + 2 * k_bytes;
  uint8_t* sP = sV + 2 * v_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + NT * (LP_BQ * LP_BK * 2));
  uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = bars + 3, *v_full = bars + 5, *v_empty = bars + 7;
  uint64_t *bar_s = bars + 9, *bar_p = bar_s + 2 * NT, *bar_o = bar_p + NT;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bar_o + NT);
  int* s_tile = reinterpret_cast<int*>(tmem_holder + 2);  // query start, first row, queries, key start, keys, found

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y, kvh = head / p.kv_group;   // of the values; keys: kh
  const int kh = PAIR ? 2 * kvh : p.key_maps > 1 ? 2 * kvh + (head & 1) : kvh;
  if (threadIdx.x == 0) {
    int t = blockIdx.x, found = 0, qs = 0, q0 = 0, nq = 0, ks = 0, nk = 0;
    for (int s = 0; s < p.num_seqs; ++s) {
      const int a = p.cu_q[s], b = p.cu_q[s + 1], nt = (b - a + RT * LP_BQ - 1) / (RT * LP_BQ);
      if (t < nt) {
        qs = a; nq = b - a; q0 = (nt - 1 - t) * RT * LP_BQ; ks = p.cu_k[s]; nk = p.cu_k[s + 1] - ks; found = 1;
        break;
      }
      t -= nt;
    }
    s_tile[0] = qs; s_tile[1] = q0; s_tile[2] = nq; s_tile[3] = ks; s_tile[4] = nk; s_tile[5] = found;
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    for (int i = 0; i < 2 * NT; ++i) mbar_init(&bar_s[i], 1);
    for (int i = 0; i < NT; ++i) {
      mbar_init(&bar_p[i], 4);
      mbar_init(&bar_o[i], 1);
    }
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, static_cast<uint32_t>(p.tmem_cols));
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  const int seq_q = s_tile[0], q0 = s_tile[1], nq = s_tile[2], seq_k = s_tile[3], nk = s_tile[4];
  const bool valid = s_tile[5] != 0;
  const int off = nk - nq;  // position of query row 0 among the sequence's keys
  auto first_key = [&](int pos) { return p.window > 0 ? max(0, pos - p.window + 1) : p.chunk > 0 ? pos / p.chunk * p.chunk : 0; };
  // key blocks: entry j of the list holds keys [block_at(j) * 64, + 64); tile t uses j in [ja[t], jz[t]). Blocks of kept keys in front
  // of the window's come first; every tile walks the list from its start then.
  int jb0 = 0, nkeep = 0, ja[NT], jz[NT], nblk = 0;
#pragma unroll
  for (int t = 0; t < NT; ++t) {
    const int r0 = q0 + (PAIR ? 0 : t) * LP_BQ;
    const int lo = first_key(r0 + off);
    if (t == 0) {
      jb0 = lo / LP_BK;
      nkeep = min((p.keep + LP_BK - 1) / LP_BK, jb0);
    }
    const bool act = valid && r0 < nq;
    ja[t] = act && p.keep == 0 ? lo / LP_BK - jb0 : 0;
    jz[t] = act ? min(min(r0 + LP_BQ, nq) - 1 + off, nk - 1) / LP_BK - jb0 + 1 + nkeep : 0;
    nblk = max(nblk, jz[t]);
  }
  auto block_at = [&](int j) { return j < nkeep ? j : jb0 + j - nkeep; };
  const uint32_t tm_o = NT * 2 * LP_BK;

  if (warp == 0) {
    if (lane == 0 && valid) {
      mbar_expect_tx(q_full, static_cast<uint32_t>(NT * q_bytes));
      for (int t = 0; t < NT; ++t) {
        const int row = seq_q + q0 + (PAIR ? 0 : t) * LP_BQ;
        for (int c = 0; c < p.pu; ++c) tma_load_3d(sQ + t * q_bytes + c * (LP_BQ * 128), &tm_qu, q_full, 64 * c, PAIR ? 2 * head + t : head, row);
        for (int c = 0; c < p.pr; ++c) tma_load_3d(sQ + t * q_bytes + (p.pu + c) * (LP_BQ * 128), &tm_qr, q_full, 64 * c, head, row);
      }
      for (int j = 0; j < nblk; ++j) {
        const int st = j & 1, row = seq_k + block_at(j) * LP_BK;
        const uint32_t ph = ((j >> 1) & 1) ^ 1;
        if (!mbar_wait(&k_empty[st], ph)) { atomicExch(p.status, ST_TIMEOUT_PRODUCER); break; }
        mbar_expect_tx(&k_full[st], static_cast<uint32_t>(k_bytes));
        for (int c = 0; c < p.pu; ++c) tma_load_3d(sK + st * k_bytes + c * (LP_BK * 128), &tm_ku, &k_full[st], 64 * c, kh, row);
        if constexpr (PAIR)
          for (int c = 0; c < p.pu; ++c) tma_load_3d(sK + st * k_bytes + map_bytes + c * (LP_BK * 128), &tm_ku, &k_full[st], 64 * c, kh + 1, row);
        for (int c = 0; c < p.pr; ++c) tma_load_2d(sK + st * k_bytes + (p.pu + c) * (LP_BK * 128), &tm_kr, &k_full[st], 64 * c, row);
        if (!mbar_wait(&v_empty[st], ph)) { atomicExch(p.status, ST_TIMEOUT_PRODUCER); break; }
        mbar_expect_tx(&v_full[st], static_cast<uint32_t>(v_bytes));
        for (int c = 0; c < p.pv; ++c) tma_load_3d(sV + st * v_bytes + c * (LP_BK * 128), &tm_v, &v_full[st], 64 * c, kvh, row);
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && valid) {
      const uint32_t idesc_s = make_idesc_f16(LP_BQ, LP_BK, false, false), idesc_o = make_idesc_f16(LP_BQ, p.pv * 64, false, true);
      bool ok = mbar_wait(q_full, 0);
      auto issue_s = [&](int j) {
        const int st = j & 1;
        if (!mbar_wait(&k_full[st], (j >> 1) & 1)) return false;
        tc_fence_after();
#pragma unroll
        for (int t = 0; t < NT; ++t) {
          if (j < ja[t] || j >= jz[t]) continue;
          const int jj = j - ja[t];
          const uint32_t d = tmem_base + (t * 2 + (jj & 1)) * LP_BK;
          const uint32_t aq = smem_u32(sQ + t * q_bytes), bk = smem_u32(sK + st * k_bytes + (PAIR ? t * map_bytes : 0));
          for (int k = 0; k < p.su; ++k)
            tc_mma_f16_ss(d, make_smem_desc_sw128(aq + (k >> 2) * (LP_BQ * 128) + (k & 3) * 32, 16, 1024),
                          make_smem_desc_sw128(bk + (k >> 2) * (LP_BK * 128) + (k & 3) * 32, 16, 1024), idesc_s, k > 0 ? 1u : 0u);
          const uint32_t ar = aq + p.pu * (LP_BQ * 128), br = bk + p.pu * (LP_BK * 128);
          for (int k = 0; k < p.sr; ++k)
            tc_mma_f16_ss(d, make_smem_desc_sw128(ar + (k >> 2) * (LP_BQ * 128) + (k & 3) * 32, 16, 1024),
                          make_smem_desc_sw128(br + (k >> 2) * (LP_BK * 128) + (k & 3) * 32, 16, 1024), idesc_s, 1u);
          tc_commit(&bar_s[t * 2 + (jj & 1)]);
        }
        tc_commit(&k_empty[st]);
        return true;
      };
      if (ok && nblk > 0) ok = issue_s(0);
      for (int j = 0; j < nblk && ok; ++j) {
        if (j + 1 < nblk) ok = issue_s(j + 1);
        if (!ok) break;
        const int st = j & 1;
        if (!mbar_wait(&v_full[st], (j >> 1) & 1)) { ok = false; break; }
#pragma unroll
        for (int t = 0; t < NT; ++t) {
          if (j < ja[t] || j >= jz[t]) continue;
          const int jj = j - ja[t];
          if (!mbar_wait(&bar_p[t], jj & 1)) { ok = false; break; }
          tc_fence_after();
          const uint32_t ap = smem_u32(sP + t * (LP_BQ * LP_BK * 2)), bv = smem_u32(sV + st * v_bytes);
#pragma unroll
          for (int k = 0; k < LP_BK / 16; ++k)
            tc_mma_f16_ss(tmem_base + tm_o + t * p.pv * 64, make_smem_desc_sw128(ap + k * 32, 16, 1024),
                          make_smem_desc_sw128(bv + k * 2048, LP_BK * 128, 1024), idesc_o, (jj > 0 || k > 0) ? 1u : 0u);
          tc_commit(&bar_o[t]);
        }
        if (!ok) break;
        tc_commit(&v_empty[st]);
      }
      if (!ok) atomicExch(p.status, ST_TIMEOUT_MMA);
    }
  } else {
    const int t = (warp - 2) >> 2;
    int a = 0, z = 0;
#pragma unroll
    for (int u = 0; u < NT; ++u)
      if (u == t) { a = ja[u]; z = jz[u]; }
    const int n = z - a;
    if (n > 0) {
      const int quad = warp & 3, r = quad * 32 + lane;
      const int row = q0 + (PAIR ? 0 : t) * LP_BQ + r;      // row inside the sequence's queries
      const int pos = row + off;               // its position among the keys
      const int tile_lo = q0 + (PAIR ? 0 : t) * LP_BQ + off, tile_hi = tile_lo + LP_BQ - 1;
      const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
      const uint32_t o_base = tmem_base + tm_o + t * p.pv * 64 + lane_off;
      const int row_first = first_key(pos);    // without a window
      float m_run = -INFINITY, l_run = 0.f;
      if (p.sink != nullptr) { m_run = __bfloat162float(p.sink[head]) * 1.4426950408889634f; l_run = 1.f; }
      bool ok = true;
      for (int jj = 0; jj < n; ++jj) {
        if (!mbar_wait(&bar_s[t * 2 + (jj & 1)], (jj >> 1) & 1)) { ok = false; break; }
        tc_fence_after();
        uint32_t x0[32], x1[32];
        tmem_ld_32x32(tmem_base + (t * 2 + (jj & 1)) * LP_BK + lane_off, x0);
        tmem_ld_32x32(tmem_base + (t * 2 + (jj & 1)) * LP_BK + 32 + lane_off, x1);
        tmem_ld_wait();
        const int col0 = block_at(a + jj) * LP_BK;
        const bool need_mask = col0 + LP_BK - 1 > tile_lo || (p.window > 0 && tile_hi - col0 >= p.window) || (p.chunk > 0 && first_key(tile_hi) > col0);
        // visible: first_c <= c <= last_c, or c < keep_c and c <= last_c
        const int last_c = pos - col0, first_c = p.window > 0 ? pos - p.window + 1 - col0 : row_first - col0, keep_c = p.keep - col0;
        float mx = -INFINITY;
        if constexpr (CAP) {
          float most = 0.f;
#pragma unroll
          for (int c = 0; c < 32; ++c) most = fmaxf(most, fmaxf(fabsf(__uint_as_float(x0[c])), fabsf(__uint_as_float(x1[c]))));
          if (__any_sync(0xffffffffu, most > p.cap_near)) {   // beyond the polynomial: the exponential form
            auto cap = [&](uint32_t& x) {
              const float z = fminf(__uint_as_float(x) * p.cap_z, 20.f);
              x = __float_as_uint(p.cap_log2 * (1.f - __fdividef(2.f, 1.f + exp2f(z * 2.8853900817779268f))));
            };
#pragma unroll
            for (int c = 0; c < 32; ++c) { cap(x0[c]); cap(x1[c]); }
          } else {
            const uint64_t a0 = both2(p.cap_poly[0]), a1 = both2(p.cap_poly[1]), a2 = both2(p.cap_poly[2]), a3 = both2(p.cap_poly[3]), a4 = both2(p.cap_poly[4]);
            auto cap = [&](uint32_t& x, uint32_t& y) {
              const uint64_t z = pack2(x, y), s = mul2(z, z);
              unpack2(mul2(z, fma2(s, fma2(s, fma2(s, fma2(s, a4, a3), a2), a1), a0)), x, y);
            };
#pragma unroll
            for (int c = 0; c < 32; c += 2) { cap(x0[c], x0[c + 1]); cap(x1[c], x1[c + 1]); }
          }
        } else {
          const uint64_t f = both2(p.scale_log2);
#pragma unroll
          for (int c = 0; c < 32; c += 2) {
            unpack2(mul2(pack2(x0[c], x0[c + 1]), f), x0[c], x0[c + 1]);
            unpack2(mul2(pack2(x1[c], x1[c + 1]), f), x1[c], x1[c + 1]);
          }
        }
        if (need_mask) {
#pragma unroll
          for (int c = 0; c < 32; ++c) {
            if (c > last_c || (c < first_c && c >= keep_c)) x0[c] = 0xff800000u;
            if (c + 32 > last_c || (c + 32 < first_c && c + 32 >= keep_c)) x1[c] = 0xff800000u;
          }
        }
#pragma unroll
        for (int c = 0; c < 32; ++c) mx = fmaxf(mx, fmaxf(__uint_as_float(x0[c]), __uint_as_float(x1[c])));
        float alpha = 1.f;
        const bool grow = mx > m_run + 8.f;   // also the first visible key of a row without a sink
        if (grow) {
          alpha = exp2f(m_run - mx);          // 0 from an empty row
          m_run = mx;
          l_run *= alpha;
        }
        const uint64_t minus_m = both2(m_run == -INFINITY ? 0.f : -m_run);
        uint64_t sum = 0;
        uint32_t pk[32];
        auto weight = [&](uint32_t a, uint32_t b) {
          uint32_t u, v;
          unpack2(add2(pack2(a, b), minus_m), u, v);
          const float e0 = exp2f(__uint_as_float(u)), e1 = exp2f(__uint_as_float(v));
          sum = add2(sum, pack2(__float_as_uint(e0), __float_as_uint(e1)));
          return pack_bf16x2(e0, e1);
        };
#pragma unroll
        for (int c = 0; c < 32; c += 2) {
          pk[c >> 1] = weight(x0[c], x0[c + 1]);
          pk[16 + (c >> 1)] = weight(x1[c], x1[c + 1]);
        }
        uint32_t s_lo, s_hi;
        unpack2(sum, s_lo, s_hi);
        l_run += __uint_as_float(s_lo) + __uint_as_float(s_hi);
        if (jj > 0) {
          // P and O are in use by the previous block's product until bar_o
          if (!mbar_wait(&bar_o[t], (jj - 1) & 1)) { ok = false; break; }
          tc_fence_after();
          if (__any_sync(0xffffffffu, grow)) {
            for (int c = 0; c < p.pv * 2; ++c) {
              uint32_t o[32];
              tmem_ld_32x32(o_base + c * 32, o);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
              tmem_st_32x32(o_base + c * 32, o);
            }
            tmem_st_wait();
          }
        }
        uint8_t* prow = sP + t * (LP_BQ * LP_BK * 2) + r * 128;
#pragma unroll
        for (int ch = 0; ch < 8; ++ch)
          *reinterpret_cast<uint4*>(prow + ((ch ^ (r & 7)) << 4)) = make_uint4(pk[ch * 4], pk[ch * 4 + 1], pk[ch * 4 + 2], pk[ch * 4 + 3]);
        fence_proxy_async_smem();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bar_p[t]);
      }
      if (ok) ok = mbar_wait(&bar_o[t], (n - 1) & 1);
      if (!ok && lane == 0) atomicExch(p.status, ST_TIMEOUT_EPILOGUE);
      if constexpr (PAIR) {
        // every softmax warp comes here, also one that gave up: both maps walk the same blocks
        tc_fence_after();
        pair_epilogue(p, smem_raw, tmem_base + tm_o + lane_off, t, r, lane, l_run > 0.f ? 1.f / l_run : 0.f, ok && row < nq,
                      static_cast<long long>(seq_q) + row, head);
      } else if (ok) {
        tc_fence_after();
        const bool row_ok = row < nq;
        const long long tok = static_cast<long long>(seq_q) + row;
        float f = l_run > 0.f ? 1.f / l_run : 0.f;
        if (p.gate != nullptr && row_ok) f /= 1.f + __expf(-p.gate[tok * p.ldg + head]);
        for (int c = 0; c < p.pv * 2; ++c) {
          uint32_t o[32];
          tmem_ld_32x32(o_base + c * 32, o);
          tmem_ld_wait();
          if (row_ok) {
            __nv_bfloat16* dst = p.out + tok * p.ldo + static_cast<long long>(head) * p.dv + c * 32;
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
              if (c * 32 + i < p.dv) {
                uint4 v;
                v.x = pack_bf16x2(__uint_as_float(o[i]) * f, __uint_as_float(o[i + 1]) * f);
                v.y = pack_bf16x2(__uint_as_float(o[i + 2]) * f, __uint_as_float(o[i + 3]) * f);
                v.z = pack_bf16x2(__uint_as_float(o[i + 4]) * f, __uint_as_float(o[i + 5]) * f);
                v.w = pack_bf16x2(__uint_as_float(o[i + 6]) * f, __uint_as_float(o[i + 7]) * f);
                *reinterpret_cast<uint4*>(dst + i) = v;
              }
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, static_cast<uint32_t>(p.tmem_cols));
  }
}

static int latent_prefill_smem(int nt, int qp, int pv, int maps = 1) {
  return nt * qp * LP_BQ * 128 + 2 * maps * qp * LP_BK * 128 + 2 * pv * LP_BK * 128 + nt * LP_BQ * LP_BK * 2 + 192;
}

}  // namespace vb

using namespace vb;

// Returns -1 for sizes, strides and alignments it does not serve. Tk: key rows.
extern "C" int vb_latent_prefill(const VbLatentAttn* a, int Tk, cudaStream_t stream) {
  const int pu = (a->du + 63) / 64, pr = (a->dr + 63) / 64, pv = (a->dv + 63) / 64;
  auto mis = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) != 0; };
  if (a->du < 8 || a->dr < 0 || a->du % 8 || a->dr % 8 || a->dv % 8 || a->hq % 8 || a->ldq % 8 || a->ku_head % 8 || a->ku_row % 8 || a->kr_row % 8 ||
      a->v_head % 8 || a->v_row % 8 || a->ldo % 8 || mis(a->q) || mis(a->ku) || (a->dr > 0 && mis(a->kr)) || mis(a->v) || mis(a->out) || pv > 4)
    return -1;
  const int limit = 232448, qp = pu + pr, maps = a->maps > 1 ? a->maps : 1;
  if (maps > 1 && (maps != 2 || pv > 2 || pr > 0 || a->gate != nullptr || a->sink != nullptr || a->softcap > 0.f || latent_prefill_smem(2, qp, pv, 2) > limit)) return -1;
  const bool pair = pv <= 2 && 2 * (latent_prefill_smem(1, qp, pv) + 1024) <= 228 * 1024;   // two CTAs of one tile (and 256 TMEM columns each)
  const int nt = maps == 2 ? 2 : (!pair && pv <= 2 && latent_prefill_smem(2, qp, pv) <= limit) ? 2 : 1;
  const int smem = latent_prefill_smem(nt, qp, pv, maps), rows_cta = (maps == 2 ? 1 : nt) * LP_BQ;
  if (smem > limit) return -1;
  const auto bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const auto sw = CU_TENSOR_MAP_SWIZZLE_128B;
  CUtensorMap tqu, tqr, tku, tkr, tv;
  const char* qr = reinterpret_cast<const char*>(a->q) + 2 * a->du;
  if (a->dr > 0 && mis(qr)) return -1;
  // a PAIR's heads count once; split maps are heads of their own, two of which share values
  const int key_maps = maps == 2 || a->split_maps ? 2 : 1, kv_group = (a->kv_group > 1 ? a->kv_group : 1) * (a->split_maps ? 2 : 1);
  const int kv_heads = a->H / maps / kv_group;
  if (!make_tmap_3d(&tqu, a->q, bf, 2, a->du, a->H, a->T, a->hq, a->ldq, 64, 1, LP_BQ, sw) ||
      !make_tmap_3d(&tku, a->ku, bf, 2, a->du, kv_heads * key_maps, Tk, a->ku_head, a->ku_row, 64, 1, LP_BK, sw) ||
      !make_tmap_3d(&tv, a->v, bf, 2, a->dv, kv_heads, Tk, a->v_head, a->v_row, 64, 1, LP_BK, sw))
    return -1;
  if (a->dr > 0) {
    if (!make_tmap_3d(&tqr, qr, bf, 2, a->dr, a->H, a->T, a->hq, a->ldq, 64, 1, LP_BQ, sw) ||
        !make_tmap_2d(&tkr, a->kr, bf, 2, Tk, a->dr, a->kr_row, 64, LP_BK, sw))
      return -1;
  } else {          // never used
    tqr = tqu;
    tkr = tku;
  }
  static int* status = nullptr;
  if (status == nullptr) cudaGetSymbolAddress(reinterpret_cast<void**>(&status), g_latent_prefill_status);
  LatentPrefillParams p{};
  p.cu_q = a->cu_q; p.cu_k = a->cu_k; p.num_seqs = a->B; p.dv = a->dv; p.window = a->window; p.keep = a->window > 0 ? a->keep_first : 0; p.chunk = a->chunk; p.kv_group = kv_group; p.pu = pu; p.pr = pr; p.pv = pv;
  p.su = (a->du + 15) / 16; p.sr = (a->dr + 15) / 16;
  p.sink = reinterpret_cast<const __nv_bfloat16*>(a->sink); p.gate = a->gate; p.ldg = a->ldg;
  p.out = reinterpret_cast<__nv_bfloat16*>(a->out); p.ldo = a->ldo; p.scale_log2 = a->scale * 1.4426950408889634f; p.status = status;
  if (a->softcap > 0.f) {
    // tanh(z) = z (c0 + c1 z^2 + ...) for |z| <= 1/2: interpolated at the five Chebyshev nodes of z^2 in [0, 1/4], relative error 1.4e-8
    const double c[5] = {0.9999999867573895, -0.3333306794442257, 0.13324750504795058, -0.05298423882896009, 0.01713134443244478};
    const double z = static_cast<double>(a->scale) / a->softcap;
    p.cap_z = static_cast<float>(z);
    p.cap_log2 = a->softcap * 1.4426950408889634f;
    p.cap_near = static_cast<float>(0.5 / (z > 0 ? z : -z));
    double f = a->softcap * 1.4426950408889634 * z;
    for (int i = 0; i < 5; ++i, f *= z * z) p.cap_poly[i] = static_cast<float>(c[i] * f);
  }
  p.tmem_cols = 128;
  while (p.tmem_cols < nt * (2 * LP_BK + pv * 64)) p.tmem_cols *= 2;
  p.diff_vec = reinterpret_cast<const __nv_bfloat16*>(a->diff_vec); p.du = a->du; p.key_maps = key_maps; p.diff = a->diff; p.eps = a->eps;
  const dim3 grid((a->T + rows_cta - 1) / rows_cta + a->B, a->H / maps);
  auto go = [&](auto kern) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, limit);
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<grid, 64 + 128 * nt, smem, stream>>>(tqu, tqr, tku, tkr, tv, p);
    return static_cast<int>(cudaGetLastError());
  };
  if (maps == 2) return go(latent_prefill_kernel<2, false, true>);
  if (a->softcap > 0.f) return nt == 2 ? go(latent_prefill_kernel<2, true, false>) : go(latent_prefill_kernel<1, true, false>);
  return nt == 2 ? go(latent_prefill_kernel<2, false, false>) : go(latent_prefill_kernel<1, false, false>);
}

extern "C" int vb_latent_prefill_status() {
  int h = 0;
  if (cudaMemcpyFromSymbol(&h, g_latent_prefill_status, sizeof(int)) != cudaSuccess) return -1;
  if (h != 0) {
    const int z = 0;
    cudaMemcpyToSymbol(g_latent_prefill_status, &z, sizeof(int));
  }
  return h;
}
