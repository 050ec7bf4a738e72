// Decode-step grouped-query attention over the paged cache of a mixer stack: one CTA = (sequence, key / value head and up to 16
// of its query heads [, key split]).
//
// A cached row is [keys of all heads | values of all heads], with query / key and value sizes of their own. Tiles of 64 tokens
// of one head are streamed once by TMA (128B swizzle, panels of 64 columns) into a three-stage shared-memory ring; the query
// heads are the M dimension of m16n8k16 MMAs: like every decode attention the kernel is bound by the stream, not by the
// tensor pipe. Each of four warps owns 16 of a tile's tokens and keeps its own online softmax; warps and key splits are merged
// at the end, where the sink (one more score without a value) joins the denominator. Scores may be capped
// (cap * tanh(score / cap)). Only the tiles of the window (or chunk) and of the kept first tokens are loaded. Differential attention: the
// two key maps of a head are one key of twice the size, a query row is zero in the other map's half, so the stream is read once; the
// merge forms the normed difference. Compiled without fast math.
#include "mixer_epilogue.cuh"
#include "mixers.h"
#include "mixer_common.cuh"
#include "tcgen05_common.cuh"

#include <math.h>

namespace vb {

constexpr int GD_TOK = 64, GD_STAGES = 3, GD_THREADS = 128, GD_HEADS = 16;

struct GroupedDecodeParams {
  const __nv_bfloat16* q;   // [S, H, dim]
  long long ldq;
  int hq;
  const int* block_table;
  int max_blocks, block_size, box_rows;
  long long num_blocks;
  const int* ctx_len;
  const __nv_bfloat16* sink;
  __nv_bfloat16* out;       // [S, H, vdim]
  float* part_o;            // [S, H, nsplit, vdim] when nsplit > 1
  float* part_ml;           // [S, H, nsplit, 2]
  int H, share, chunks, dim, vdim, window, keep, chunk, nsplit;   // chunks: groups of 16 query heads per key head
  float scale_log2, cap_z, cap_log2;
  // differential attention: H and share count maps, dim spans both key maps of a head; a query row fills its map's half
  int maps, map_dim;
  const __nv_bfloat16* diff_vec;   // four vectors of map_dim
  float diff, eps;
  int* status;
};

__device__ int g_grouped_decode_status[1];

__device__ __forceinline__ void gd_ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void gd_ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void gd_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// lambda = exp(x0 . x1) - exp(x2 . x3) + diff, every lane of the warp gets it
__device__ __forceinline__ float gd_lambda(const __nv_bfloat16* x, int n, float diff) {
  float a = 0.f, b = 0.f;
  for (int i = threadIdx.x & 31; i < n; i += 32) {
    a = fmaf(__bfloat162float(x[i]), __bfloat162float(x[n + i]), a);
    b = fmaf(__bfloat162float(x[2 * n + i]), __bfloat162float(x[3 * n + i]), b);
  }
  return expf(warp_sum(a)) - expf(warp_sum(b)) + diff;
}

template <int PK, int PV>
struct GDSmem {
  static constexpr int K_BYTES = PK * GD_TOK * 128, STAGE = K_BYTES + PV * GD_TOK * 128;
  static constexpr int MERGE_LD = PV * 64 + 2;
  static constexpr int MERGE = 4 * GD_HEADS * MERGE_LD * 4;   // four warps' results, in the ring's place
  static constexpr int RING = (GD_STAGES * STAGE > MERGE ? GD_STAGES * STAGE : (MERGE + 1023) / 1024 * 1024);
  static constexpr int QPITCH = PK * 128 + 16;                // shifted banks per head
  static constexpr int OFF_BAR = RING + (GD_HEADS * QPITCH + 15) / 16 * 16;
  static constexpr int TOTAL = OFF_BAR + 64 + 1024;
};

template <int PK, int PV>
__global__ void __launch_bounds__(GD_THREADS, GDSmem<PK, PV>::TOTAL <= 113 * 1024 ? 2 : 1)
grouped_decode_kernel(const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v, const GroupedDecodeParams p) {
  using L = GDSmem<PK, PV>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem + L::RING;
  float* sM = reinterpret_cast<float*>(smem);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);
  uint64_t* empty = full + GD_STAGES;

  const int b = blockIdx.x, kvh = blockIdx.y / p.chunks, split = blockIdx.z;
  const int h_in = (blockIdx.y % p.chunks) * GD_HEADS;        // first of this CTA's heads inside the group
  const int h0 = kvh * p.share + h_in, nh = min(GD_HEADS, p.share - h_in);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3, r8 = lane & 7;
  const int len = min(p.ctx_len[b], p.max_blocks * p.block_size);
  const int first = (p.window > 0 && len > p.window) ? len - p.window : (p.chunk > 0 && len > 0) ? (len - 1) / p.chunk * p.chunk : 0;
  const int tile_a = first / GD_TOK, tile_b = (len + GD_TOK - 1) / GD_TOK;
  // the list of tiles: those of the kept tokens that lie in front of the window's, then the window's
  const int nkeep = min((p.keep + GD_TOK - 1) / GD_TOK, tile_a), listed = nkeep + max(0, tile_b - tile_a);
  const int per = (listed + p.nsplit - 1) / p.nsplit;
  const int t0 = split * per, n = max(0, min(listed, t0 + per) - t0);
  auto tile_at = [&](int i) { return t0 + i < nkeep ? t0 + i : tile_a + t0 + i - nkeep; };
  const int* bt = p.block_table + static_cast<long long>(b) * p.max_blocks;

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
    for (int s = 0; s < GD_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 4);
    }
    mbar_fence_init();
  }
  for (int i = threadIdx.x; i < GD_HEADS * PK * 8; i += GD_THREADS) {
    const int g = i / (PK * 8), c = i % (PK * 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    const int at = c * 8 - (p.maps > 1 && (g & 1) ? p.map_dim : 0);   // heads start at even rows
    if (g < nh && at >= 0 && at < p.map_dim) v = *reinterpret_cast<const uint4*>(p.q + b * p.ldq + static_cast<long long>(h0 + g) * p.hq + at);
    *reinterpret_cast<uint4*>(sQ + g * L::QPITCH + c * 16) = v;
  }
  __syncthreads();

  auto issue = [&](int i) {   // tile t0 + i into stage i % GD_STAGES (thread 0 only)
    const int s = i % GD_STAGES, tok = tile_at(i) * GD_TOK;
    uint8_t* dst = smem + s * L::STAGE;
    mbar_expect_tx(&full[s], L::STAGE);
    for (int r = 0; r < GD_TOK; r += p.box_rows) {
      // rows past the context re-read its last box: they are masked below
      const int at = min(tok + r, (len - 1) / p.box_rows * p.box_rows);
      const int blk = max(0, min(bt[at / p.block_size], static_cast<int>(p.num_blocks) - 1));
#pragma unroll
      for (int c = 0; c < PK; ++c) tma_load_4d(dst + c * (GD_TOK * 128) + r * 128, &tm_k, &full[s], c * 64, kvh, at % p.block_size, blk);
#pragma unroll
      for (int c = 0; c < PV; ++c) tma_load_4d(dst + L::K_BYTES + c * (GD_TOK * 128) + r * 128, &tm_v, &full[s], c * 64, kvh, at % p.block_size, blk);
    }
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < min(n, GD_STAGES); ++i) issue(i);

  uint32_t qa[PK * 4][4];
#pragma unroll
  for (int k = 0; k < PK * 4; ++k) gd_ldsm_x4(qa[k], smem_u32(sQ) + ((mi & 1) * 8 + r8) * L::QPITCH + k * 32 + (mi >> 1) * 16);
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  float o[PV * 8][4];
#pragma unroll
  for (int j = 0; j < PV * 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;

  bool ok = true;
  const int tw = warp * 16;   // this warp's tokens inside a tile
  for (int i = 0; i < n; ++i) {
    const int s = i % GD_STAGES;
    if (!__all_sync(0xffffffffu, mbar_wait(&full[s], (i / GD_STAGES) & 1))) { ok = false; break; }
    const uint32_t kbase = smem_u32(smem + s * L::STAGE), vbase = kbase + L::K_BYTES;
    float sc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      const int tok = tw + nb * 8 + r8;
#pragma unroll
      for (int k2 = 0; k2 < PK * 2; ++k2) {   // two k steps per ldmatrix.x4
        const int dc = k2 * 4 + mi;           // 16-byte chunk along the key
        uint32_t kb[4];
        gd_ldsm_x4(kb, kbase + (dc >> 3) * (GD_TOK * 128) + tok * 128 + (((dc & 7) ^ (tok & 7)) << 4));
        gd_mma(sc[nb], qa[2 * k2], kb[0], kb[1]);
        gd_mma(sc[nb], qa[2 * k2 + 1], kb[2], kb[3]);
      }
    }
    // rows: heads lane / 4 and + 8; columns: tokens 8 nb + 2 (lane % 4) and + 1
    const int tok_base = tile_at(i) * GD_TOK + tw + (lane & 3) * 2;
    float alpha[2];
    uint32_t pa[4];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float v[4];
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = tok_base + nb * 8 + e;
          const float x = sc[nb][h * 2 + e];
          const float y = p.cap_log2 > 0.f ? p.cap_log2 * tanh_full(x * p.cap_z) : x * p.scale_log2;
          v[nb * 2 + e] = ((t >= first || t < p.keep) && t < len) ? y : -INFINITY;
        }
      float mx = fmaxf(fmaxf(v[0], v[1]), fmaxf(v[2], v[3]));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float mn = fmaxf(m_run[h], mx);
      const float mu = mn == -INFINITY ? 0.f : mn;
      alpha[h] = mn == -INFINITY ? 1.f : exp2f(m_run[h] - mn);
      m_run[h] = mn;
      const float e0 = exp2f(v[0] - mu), e1 = exp2f(v[1] - mu), e2 = exp2f(v[2] - mu), e3 = exp2f(v[3] - mu);
      l_run[h] = l_run[h] * alpha[h] + (e0 + e1) + (e2 + e3);   // this thread's tokens only
      pa[h] = pack_bf16x2(e0, e1);
      pa[2 + h] = pack_bf16x2(e2, e3);
    }
    const int tok = tw + (mi & 1) * 8 + r8;
    const bool grew = __any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f);
#pragma unroll
    for (int j2 = 0; j2 < PV * 4; ++j2) {   // two 8-column blocks per ldmatrix.x4.trans
      const int dc = j2 * 2 + (mi >> 1);
      uint32_t vb[4];
      gd_ldsm_x4_t(vb, vbase + (dc >> 3) * (GD_TOK * 128) + tok * 128 + (((dc & 7) ^ (tok & 7)) << 4));
#pragma unroll
      for (int q2 = 0; q2 < 2; ++q2) {
        float(&oo)[4] = o[2 * j2 + q2];
        if (grew) { oo[0] *= alpha[0]; oo[1] *= alpha[0]; oo[2] *= alpha[1]; oo[3] *= alpha[1]; }
        gd_mma(oo, pa, vb[2 * q2], vb[2 * q2 + 1]);
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[s]);
    if (threadIdx.x == 0 && i + GD_STAGES < n) {
      if (mbar_wait(&empty[s], (i / GD_STAGES) & 1)) issue(i + GD_STAGES);
      else atomicExch(p.status, 2);   // the consumers' next wait on this stage then runs out too
    }
    __syncwarp();
  }
  if (!ok && lane == 0) atomicExch(p.status, 1);

  // merge the four warps: row (warp, head) = [o | m, l]; every tile has been waited for, so the ring is idle
  __syncthreads();
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    float l = l_run[h];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    float* row = sM + (warp * GD_HEADS + (lane >> 2) + 8 * h) * L::MERGE_LD;
#pragma unroll
    for (int j = 0; j < PV * 8; ++j) {
      row[j * 8 + (lane & 3) * 2] = o[j][2 * h];
      row[j * 8 + (lane & 3) * 2 + 1] = o[j][2 * h + 1];
    }
    if ((lane & 3) == 0) {
      row[PV * 64] = m_run[h];
      row[PV * 64 + 1] = l;
    }
  }
  __syncthreads();
  if (p.maps > 1 && p.nsplit == 1) {   // a warp per head: both maps merged, their difference normed
    const float lam = gd_lambda(p.diff_vec, p.map_dim, p.diff);
    for (int hh = warp; hh < nh / 2; hh += GD_THREADS / 32) {
      float f[2][4];
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const float* row = sM + (2 * hh + m) * L::MERGE_LD;
        float M = -INFINITY, l = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) M = fmaxf(M, row[w * GD_HEADS * L::MERGE_LD + PV * 64]);
#pragma unroll
        for (int w = 0; w < 4; ++w) {
          const float* rw = row + w * GD_HEADS * L::MERGE_LD;
          f[m][w] = rw[PV * 64] == -INFINITY ? 0.f : exp2f(rw[PV * 64] - M);
          l += rw[PV * 64 + 1] * f[m][w];
        }
        const float s = len > 0 && l > 0.f ? (m == 0 ? 1.f : -lam) / l : 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) f[m][w] *= s;
      }
      float z[PV * 2], ss = 0.f;
#pragma unroll
      for (int i = 0; i < PV * 2; ++i) {
        const int d = i * 32 + lane;
        z[i] = 0.f;
        if (d < p.vdim) {
#pragma unroll
          for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int w = 0; w < 4; ++w) z[i] += sM[(w * GD_HEADS + 2 * hh + m) * L::MERGE_LD + d] * f[m][w];
        }
        ss += z[i] * z[i];
      }
      const float r = (1.f - p.diff) / sqrtf(warp_sum(ss) / p.vdim + p.eps);
      __nv_bfloat16* o = p.out + (static_cast<long long>(b) * (p.H / 2) + h0 / 2 + hh) * p.vdim;
#pragma unroll
      for (int i = 0; i < PV * 2; ++i)
        if (i * 32 + lane < p.vdim) o[i * 32 + lane] = __float2bfloat16(z[i] * r);
    }
    return;
  }
  for (int idx = threadIdx.x; idx < nh * p.vdim; idx += GD_THREADS) {
    const int g = idx / p.vdim, d = idx % p.vdim;
    const float* row = sM + g * L::MERGE_LD;
    const bool sk = p.sink != nullptr && split == 0;
    const float m_sink = sk ? __bfloat162float(p.sink[h0 + g]) * 1.4426950408889634f : -INFINITY;
    float M = m_sink;
#pragma unroll
    for (int w = 0; w < 4; ++w) M = fmaxf(M, row[w * GD_HEADS * L::MERGE_LD + PV * 64]);
    float l = sk ? exp2f(m_sink - M) : 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float* rw = row + w * GD_HEADS * L::MERGE_LD;
      const float f = rw[PV * 64] == -INFINITY ? 0.f : exp2f(rw[PV * 64] - M);
      l += rw[PV * 64 + 1] * f;
      acc += rw[d] * f;
    }
    const long long at = static_cast<long long>(b) * p.H + h0 + g;
    if (p.nsplit == 1) {
      p.out[at * p.vdim + d] = __float2bfloat16(len > 0 && l > 0.f ? acc / l : 0.f);
    } else {
      p.part_o[(at * p.nsplit + split) * p.vdim + d] = acc;
      if (d == 0) {
        p.part_ml[(at * p.nsplit + split) * 2] = M;
        p.part_ml[(at * p.nsplit + split) * 2 + 1] = l;
      }
    }
  }
}

// Joins the key splits of one (sequence, head).
__global__ void grouped_decode_merge_kernel(const float* __restrict__ po, const float* __restrict__ ml, const int* __restrict__ ctx_len,
                                            __nv_bfloat16* __restrict__ out, int H, int nsplit, int vdim) {
  const long long row = blockIdx.x;
  const float* m = ml + row * nsplit * 2;
  float M = -INFINITY, l = 0.f;
  for (int s = 0; s < nsplit; ++s) M = fmaxf(M, m[2 * s]);
  for (int s = 0; s < nsplit; ++s) l += m[2 * s] == -INFINITY ? 0.f : exp2f(m[2 * s] - M) * m[2 * s + 1];
  const float inv = (l > 0.f && ctx_len[row / H] > 0) ? 1.f / l : 0.f;
  for (int c = threadIdx.x; c < vdim; c += blockDim.x) {
    float a = 0.f;
    for (int s = 0; s < nsplit; ++s) a += m[2 * s] == -INFINITY ? 0.f : exp2f(m[2 * s] - M) * po[(row * nsplit + s) * vdim + c];
    out[row * vdim + c] = __float2bfloat16(a * inv);
  }
}

// Joins the key splits of both maps of one (sequence, head) and finishes the difference. One warp per head.
__global__ void __launch_bounds__(32)
grouped_decode_merge_diff_kernel(const float* __restrict__ po, const float* __restrict__ ml, const int* __restrict__ ctx_len, __nv_bfloat16* __restrict__ out,
                                 const __nv_bfloat16* __restrict__ vec, int map_dim, float diff, float eps, int heads, int nsplit, int vdim) {
  const long long row = blockIdx.x;
  const int lane = threadIdx.x;
  const float lam = gd_lambda(vec, map_dim, diff);
  float z[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, ss = 0.f;
  for (int m = 0; m < 2; ++m) {
    const long long at = (row * 2 + m) * nsplit;
    float M = -INFINITY, l = 0.f;
    for (int s = 0; s < nsplit; ++s) M = fmaxf(M, ml[2 * (at + s)]);
    for (int s = 0; s < nsplit; ++s) l += ml[2 * (at + s)] == -INFINITY ? 0.f : exp2f(ml[2 * (at + s)] - M) * ml[2 * (at + s) + 1];
    const float inv = (l > 0.f && ctx_len[row / heads] > 0) ? (m == 0 ? 1.f : -lam) / l : 0.f;
    for (int s = 0; s < nsplit; ++s) {
      const float f = ml[2 * (at + s)] == -INFINITY ? 0.f : exp2f(ml[2 * (at + s)] - M) * inv;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i * 32 + lane < vdim) z[i] += f * po[(at + s) * vdim + i * 32 + lane];
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) ss += z[i] * z[i];
  const float r = (1.f - diff) / sqrtf(warp_sum(ss) / vdim + eps);
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (i * 32 + lane < vdim) out[row * vdim + i * 32 + lane] = __float2bfloat16(z[i] * r);
}

}  // namespace vb

using namespace vb;

// Key splits (0: the sizes are not served). max_keys: most keys a sequence can see.
extern "C" int vb_grouped_decode_splits(const VbLatentAttn* a, int max_keys) {
  const int maps = a->maps > 1 ? a->maps : 1, share = (a->kv_group > 1 ? a->kv_group : 1) * maps, bs = a->block_size;
  if (a->du < 8 || a->du * maps > 256 || a->du % 8 || a->dv < 8 || a->dv > 256 || a->dv % 8 || a->H % share) return 0;
  if (bs % 8 || !(bs % GD_TOK == 0 || GD_TOK % bs == 0)) return 0;
  const int ctas = a->B * (a->H / share) * ((share + GD_HEADS - 1) / GD_HEADS), tiles = (max_keys + GD_TOK - 1) / GD_TOK;
  int s = 2 * num_sms() / (ctas > 0 ? ctas : 1);
  if (s > tiles / 2) s = tiles / 2;
  return s < 1 ? 1 : (s > 32 ? 32 : s);
}

// Keys at ku (row stride ku_row inside a page, head stride ku_head; two maps are neighbours), values at v; out [B, H, dv]
// contiguous ([B, H / 2, dv] with two maps). Returns -1 for strides
// and alignments it does not serve.
extern "C" int vb_grouped_decode(const VbLatentAttn* a, long long num_blocks, int nsplit, float* part_o, float* part_ml, cudaStream_t stream) {
  if (a->B == 0) return 0;
  if (a->hq % 8 || a->ldq % 8 || a->page_stride % 8 || a->ku_row % 8 || a->ku_head % 8 || a->v_row % 8 || a->v_head % 8) return -1;
  if ((reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->ku) | reinterpret_cast<uintptr_t>(a->v)) & 15) return -1;
  GroupedDecodeParams p{};
  p.maps = a->maps > 1 ? a->maps : 1;
  p.share = (a->kv_group > 1 ? a->kv_group : 1) * p.maps;
  const int dk = a->du * p.maps;     // a head's key maps lie behind each other
  if (p.maps > 1 && (a->maps != 2 || a->ku_head != a->du || a->sink != nullptr)) return -1;
  p.chunks = (p.share + GD_HEADS - 1) / GD_HEADS;
  const int kv_heads = a->H / p.share;
  p.box_rows = a->block_size < GD_TOK ? a->block_size : GD_TOK;
  CUtensorMap tk, tv;
  const auto bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const uint64_t G = kv_heads, bs = a->block_size, nb = num_blocks, ps = a->page_stride;
  const uint32_t rows = p.box_rows;
  if (!make_tmap_4d(&tk, a->ku, bf, 2, {(uint64_t)dk, G, bs, nb}, {(uint64_t)a->ku_head * p.maps, (uint64_t)a->ku_row, ps}, {64, 1, rows, 1}, CU_TENSOR_MAP_SWIZZLE_128B) ||
      !make_tmap_4d(&tv, a->v, bf, 2, {(uint64_t)a->dv, G, bs, nb}, {(uint64_t)a->v_head, (uint64_t)a->v_row, ps}, {64, 1, rows, 1}, CU_TENSOR_MAP_SWIZZLE_128B))
    return -1;
  static int* status = nullptr;
  if (status == nullptr) cudaGetSymbolAddress(reinterpret_cast<void**>(&status), g_grouped_decode_status);
  p.q = reinterpret_cast<const __nv_bfloat16*>(a->q); p.ldq = a->ldq; p.hq = a->hq;
  p.block_table = a->block_table; p.max_blocks = a->max_blocks; p.block_size = a->block_size; p.num_blocks = num_blocks; p.ctx_len = a->ctx_len;
  p.sink = reinterpret_cast<const __nv_bfloat16*>(a->sink); p.out = reinterpret_cast<__nv_bfloat16*>(a->out); p.part_o = part_o; p.part_ml = part_ml;
  p.map_dim = a->du; p.diff_vec = reinterpret_cast<const __nv_bfloat16*>(a->diff_vec); p.diff = a->diff; p.eps = a->eps; p.chunk = a->chunk;
  p.H = a->H; p.dim = dk; p.vdim = a->dv; p.window = a->window; p.keep = a->window > 0 ? a->keep_first : 0; p.nsplit = nsplit; p.status = status;
  p.scale_log2 = a->scale * 1.4426950408889634f;
  if (a->softcap > 0.f) { p.cap_z = a->scale / a->softcap; p.cap_log2 = a->softcap * 1.4426950408889634f; }
  const dim3 grid(a->B, kv_heads * p.chunks, nsplit);
  auto go = [&](auto kern, int smem) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<grid, GD_THREADS, smem, stream>>>(tk, tv, p);
    return static_cast<int>(cudaGetLastError());
  };
  const int pk = (dk + 63) / 64, pv = (a->dv + 63) / 64;
  int rc;
  if (pk == 1 && pv == 1) rc = go(grouped_decode_kernel<1, 1>, GDSmem<1, 1>::TOTAL);
  else if (pk == 1 && pv == 2) rc = go(grouped_decode_kernel<1, 2>, GDSmem<1, 2>::TOTAL);
  else if (pk == 2 && pv == 1) rc = go(grouped_decode_kernel<2, 1>, GDSmem<2, 1>::TOTAL);
  else if (pk <= 2 && pv <= 2) rc = go(grouped_decode_kernel<2, 2>, GDSmem<2, 2>::TOTAL);
  else if (pk <= 3 && pv <= 2) rc = go(grouped_decode_kernel<3, 2>, GDSmem<3, 2>::TOTAL);
  else if (pk <= 2 && pv <= 4) rc = go(grouped_decode_kernel<2, 4>, GDSmem<2, 4>::TOTAL);
  else rc = go(grouped_decode_kernel<4, 4>, GDSmem<4, 4>::TOTAL);
  if (rc == 0 && nsplit > 1 && p.maps > 1) {
    grouped_decode_merge_diff_kernel<<<a->B * (a->H / 2), 32, 0, stream>>>(part_o, part_ml, a->ctx_len, p.out, p.diff_vec, p.map_dim, p.diff, p.eps, a->H / 2, nsplit,
                                                                           p.vdim);
    rc = static_cast<int>(cudaGetLastError());
  } else if (rc == 0 && nsplit > 1) {
    grouped_decode_merge_kernel<<<a->B * a->H, 128, 0, stream>>>(part_o, part_ml, a->ctx_len, p.out, a->H, nsplit, p.vdim);
    rc = static_cast<int>(cudaGetLastError());
  }
  return rc;
}

extern "C" int vb_grouped_decode_status() {
  int h = 0;
  if (cudaMemcpyFromSymbol(&h, g_grouped_decode_status, sizeof(int)) != cudaSuccess) return -1;
  if (h != 0) {
    const int z = 0;
    cudaMemcpyToSymbol(g_grouped_decode_status, &z, sizeof(int));
  }
  return h;
}
