// Decode-step attention in the latent space: one CTA = (sequence, one or two groups of 16 heads [, key split]).
//
// All heads read the same cached row, [latent (value and first key part) | rotated key part], so a row is streamed once per
// CTA: a producer warp brings 32-token tiles of the pages by TMA (128B swizzle, 64 columns per panel) into a shared-memory ring, and the
// 16 heads of a group of four warps are the M dimension of m16n8k16 MMAs (a 16-row sliver of work per byte: the kernel is bound by the stream, not by
// the tensor pipe, as in paged_decode_tma.cu). Per tile
//   scores   warp w takes a quarter of the row width for all 32 tokens (its query fragments stay in registers); the partial
//            scores meet in shared memory, and every warp forms the whole 16 x 32 tile of weights from them
//   softmax  running maximum starts at the sink, which adds one unit of weight and no value
//   values   warp w takes kv_rank / 4 latent columns over all 32 tokens
// so that one barrier per tile is enough.
// Only the tiles of the window and of the kept first tokens are loaded. Compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"
#include "tcgen05_common.cuh"

#include <math.h>

namespace vb {

constexpr int LD_TOK = 32, LD_HEADS = 16, LD_MAX_STAGES = 4, LD_SP = 40;  // LD_SP: row pitch of the partial scores

struct LatentDecodeParams {
  const __nv_bfloat16* q;   // [S, H, width]
  long long ldq;
  int hq;
  const int* block_table;
  int max_blocks, block_size, box_rows;
  long long num_blocks;
  const int* ctx_len;
  const __nv_bfloat16* sink;
  __nv_bfloat16* out;       // [S, H, rank]
  float* part_o;            // [S, H, nsplit, rank] when nsplit > 1
  float* part_ml;           // [S, H, nsplit, 2]
  int H, width, rank, panels, window, keep, nsplit, stages;
  float scale_log2;
  int* status;
};

__device__ int g_latent_decode_status[1];

__device__ __forceinline__ void ld_ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ld_ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ld_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// NV: 8-column value blocks per warp (rank <= 32 NV); KW: most panels (k steps of 16 per warp); NG: groups of 16 heads per CTA
template <int NV, int KW, int NG>
__global__ void __launch_bounds__(128 * NG + 32, NG == 1 ? 2 : 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm, const LatentDecodeParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int stage_bytes = p.panels * (LD_TOK * 128);
  const int qpitch = p.panels * 128 + 16;                   // bytes of one query row (shifted banks per head)
  uint8_t* sQ = smem + p.stages * stage_bytes;
  const int group = NG == 1 ? 0 : min(static_cast<int>(threadIdx.x >> 7), NG - 1);
  // per group: first the queries, then (their fragments are in registers by then) two buffers of four warps' partial scores
  const int group_bytes = max(LD_HEADS * qpitch, 2 * 4 * LD_HEADS * LD_SP * 4);
  float* sS = reinterpret_cast<float*>(sQ + group * group_bytes);
  uint64_t* full = reinterpret_cast<uint64_t*>(sQ + NG * group_bytes);  // [stages]
  uint64_t* empty = full + LD_MAX_STAGES;

  const int b = blockIdx.x, h0 = (blockIdx.y * NG + group) * LD_HEADS, split = blockIdx.z;
  const int wall = threadIdx.x >> 5, warp = wall & 3, lane = threadIdx.x & 31;
  const bool producer = wall == 4 * NG;
  sQ += group * group_bytes;
  const int len = min(p.ctx_len[b], p.max_blocks * p.block_size);
  const int nheads = max(0, min(LD_HEADS, p.H - h0));
  const int first = (p.window > 0 && len > p.window) ? len - p.window : 0;
  const int tile_a = first / LD_TOK, tile_b = (len + LD_TOK - 1) / LD_TOK;
  // the list of tiles: those of the kept tokens that lie in front of the window's, then the window's
  const int nkeep = min((p.keep + LD_TOK - 1) / LD_TOK, tile_a), listed = nkeep + max(0, tile_b - tile_a);
  const int per = (listed + p.nsplit - 1) / p.nsplit;
  const int t0 = split * per, n = max(0, min(listed, t0 + per) - t0);
  auto tile_at = [&](int i) { return t0 + i < nkeep ? t0 + i : tile_a + t0 + i - nkeep; };
  const int* bt = p.block_table + static_cast<long long>(b) * p.max_blocks;

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tm);
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 4 * NG);
    }
    mbar_fence_init();
  }
  for (int i = threadIdx.x & 127; i < LD_HEADS * p.panels * 8 && !producer; i += 128) {
    const int g = i / (p.panels * 8), c = i % (p.panels * 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (g < nheads && c * 8 < p.width) v = *reinterpret_cast<const uint4*>(p.q + b * p.ldq + static_cast<long long>(h0 + g) * p.hq + c * 8);
    *reinterpret_cast<uint4*>(sQ + g * qpitch + c * 16) = v;
  }
  __syncthreads();

  if (producer) {
    if (lane == 0) {
      for (int i = 0; i < n; ++i) {
        const int s = i % p.stages, tok = tile_at(i) * LD_TOK;
        if (i >= p.stages && !mbar_wait(&empty[s], ((i / p.stages) & 1) ^ 1)) {
          atomicExch(p.status, 2);
          break;
        }
        uint8_t* dst = smem + s * stage_bytes;
        mbar_expect_tx(&full[s], static_cast<uint32_t>(stage_bytes));
        for (int r = 0; r < LD_TOK; r += p.box_rows) {
          // rows past the context re-read its last page: they are masked below
          const int at = min(tok + r, (len - 1) / p.box_rows * p.box_rows);
          const int blk = max(0, min(bt[at / p.block_size], static_cast<int>(p.num_blocks) - 1));
          for (int c = 0; c < p.panels; ++c) tma_load_3d(dst + c * (LD_TOK * 128) + r * 128, &tm, &full[s], c * 64, at % p.block_size, blk);
        }
      }
    }
    return;   // the consumers wait for every copy before they leave
  }
  auto sync_group = [&]() { asm volatile("bar.sync %0, 128;" ::"r"(1 + group) : "memory"); };

  const int mi = lane >> 3, r8 = lane & 7;
  uint32_t qa[KW][4];
#pragma unroll
  for (int kk = 0; kk < KW; ++kk)
    if (kk < p.panels) ld_ldsm_x4(qa[kk], smem_u32(sQ) + ((mi & 1) * 8 + r8) * qpitch + (warp * p.panels + kk) * 32 + (mi >> 1) * 16);
  sync_group();                            // the queries' place becomes the partial scores'
  float m_run[2], l_run[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int hd = (lane >> 2) + 8 * h;
    const bool sk = p.sink != nullptr && split == 0 && hd < nheads;
    m_run[h] = sk ? to_f(p.sink[h0 + hd]) * 1.4426950408889634f : -INFINITY;
    l_run[h] = (sk && (lane & 3) == 0) ? 1.f : 0.f;   // per-thread share of the denominator
  }
  float o[NV][4];
#pragma unroll
  for (int j = 0; j < NV; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;

  bool ok = true;
  for (int i = 0; i < n; ++i) {
    const int s = i % p.stages;
    // a wait that runs out is recorded; the loop goes on so that every thread meets the same barriers
    if (ok && !mbar_wait(&full[s], (i / p.stages) & 1)) ok = false;
    const uint32_t kb = smem_u32(smem + s * stage_bytes);
    // ---- partial scores of all 32 tokens over this warp's k steps
    float sc[4][4] = {};
    {
      uint32_t bf[2][2][4];                // fragments one k step ahead of the products
      auto fetch = [&](int kk) {
        const int dc = (warp * p.panels + kk) * 2 + (mi & 1);
#pragma unroll
        for (int tb = 0; tb < 2; ++tb) {
          const int tok = tb * 16 + (mi >> 1) * 8 + r8;
          ld_ldsm_x4(bf[kk & 1][tb], kb + (dc >> 3) * (LD_TOK * 128) + tok * 128 + (((dc & 7) ^ (tok & 7)) << 4));
        }
      };
      fetch(0);
#pragma unroll
      for (int kk = 0; kk < KW; ++kk) {
        if (kk >= p.panels) break;
        if (kk + 1 < p.panels && kk + 1 < KW) fetch(kk + 1);
#pragma unroll
        for (int tb = 0; tb < 2; ++tb) {
          ld_mma(sc[2 * tb], qa[kk], bf[kk & 1][tb][0], bf[kk & 1][tb][1]);
          ld_mma(sc[2 * tb + 1], qa[kk], bf[kk & 1][tb][2], bf[kk & 1][tb][3]);
        }
      }
    }
    float* mine = sS + ((i & 1) * 4 + warp) * (LD_HEADS * LD_SP) + (lane >> 2) * LD_SP + (lane & 3) * 2;
#pragma unroll
    for (int nb = 0; nb < 4; ++nb) {
      *reinterpret_cast<float2*>(mine + nb * 8) = make_float2(sc[nb][0], sc[nb][1]);
      *reinterpret_cast<float2*>(mine + 8 * LD_SP + nb * 8) = make_float2(sc[nb][2], sc[nb][3]);
    }
    sync_group();
    // ---- weights: rows lane / 4 and + 8, columns 8 nb + 2 (lane % 4) and + 1
    const float* all = sS + (i & 1) * 4 * (LD_HEADS * LD_SP) + (lane >> 2) * LD_SP + (lane & 3) * 2;
    const int tok0 = tile_at(i) * LD_TOK + (lane & 3) * 2;
    float alpha[2];
    uint32_t pa[2][4];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float v[4][2], mx = -INFINITY;
#pragma unroll
      for (int nb = 0; nb < 4; ++nb) {
        float2 x = make_float2(0.f, 0.f);
#pragma unroll
        for (int w = 0; w < 4; ++w) {
          const float2 y = *reinterpret_cast<const float2*>(all + w * (LD_HEADS * LD_SP) + h * 8 * LD_SP + nb * 8);
          x.x += y.x;
          x.y += y.y;
        }
        const int t = tok0 + nb * 8;
        v[nb][0] = ((t >= first || t < p.keep) && t < len) ? x.x * p.scale_log2 : -INFINITY;
        v[nb][1] = ((t + 1 >= first || t + 1 < p.keep) && t + 1 < len) ? x.y * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, fmaxf(v[nb][0], v[nb][1]));
      }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float mn = fmaxf(mx, m_run[h]);
      const float mu = mn == -INFINITY ? 0.f : mn;
      alpha[h] = mn == -INFINITY ? 1.f : exp2f(m_run[h] - mn);
      m_run[h] = mn;
      float sum = 0.f;
#pragma unroll
      for (int nb = 0; nb < 4; ++nb) {
        const float e0 = exp2f(v[nb][0] - mu), e1 = exp2f(v[nb][1] - mu);
        sum += e0 + e1;
        pa[nb >> 1][(nb & 1) * 2 + h] = pack_bf16x2(e0, e1);
      }
      l_run[h] = l_run[h] * alpha[h] + sum;
    }
    // ---- values: this warp's columns over the 32 tokens
    if (alpha[0] != 1.f || alpha[1] != 1.f) {
#pragma unroll
      for (int j = 0; j < NV; ++j) { o[j][0] *= alpha[0]; o[j][1] *= alpha[0]; o[j][2] *= alpha[1]; o[j][3] *= alpha[1]; }
    }
    {
      uint32_t vb[2][2][4];
      auto fetch = [&](int j2) {
        const int dc = (warp * NV / 2 + j2) * 2 + (mi >> 1);
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const int tok = k * 16 + (mi & 1) * 8 + r8;
          ld_ldsm_x4_t(vb[j2 & 1][k], kb + (dc >> 3) * (LD_TOK * 128) + tok * 128 + (((dc & 7) ^ (tok & 7)) << 4));
        }
      };
      const int nj = min(NV / 2, (p.rank + 15) / 16 - warp * NV / 2);   // 16-column blocks of this warp inside the latent
      if (nj > 0) fetch(0);
#pragma unroll
      for (int j2 = 0; j2 < NV / 2; ++j2) {
        if (j2 >= nj) break;
        if (j2 + 1 < nj) fetch(j2 + 1);
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          ld_mma(o[2 * j2], pa[k], vb[j2 & 1][k][0], vb[j2 & 1][k][1]);
          ld_mma(o[2 * j2 + 1], pa[k], vb[j2 & 1][k][2], vb[j2 & 1][k][3]);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[s]);
  }
  if (!ok) atomicExch(p.status, 1);

#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int hd = (lane >> 2) + 8 * h;
    float l = l_run[h];                    // every thread holds its own tokens' share, every warp all of them
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    if (hd >= nheads) continue;
    const long long row = static_cast<long long>(b) * p.H + h0 + hd;
    const float f = p.nsplit > 1 ? 1.f : (l > 0.f && len > 0 ? 1.f / l : 0.f);
    float* po = p.nsplit > 1 ? p.part_o + (row * p.nsplit + split) * p.rank : nullptr;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int col = (warp * NV + j) * 8 + (lane & 3) * 2;
      if (col >= p.rank) continue;
      if (p.nsplit > 1) *reinterpret_cast<float2*>(po + col) = make_float2(o[j][2 * h], o[j][2 * h + 1]);
      else *reinterpret_cast<uint32_t*>(p.out + row * p.rank + col) = pack_bf16x2(o[j][2 * h] * f, o[j][2 * h + 1] * f);
    }
    if (p.nsplit > 1 && warp == 0 && (lane & 3) == 0) {
      p.part_ml[(row * p.nsplit + split) * 2] = m_run[h];
      p.part_ml[(row * p.nsplit + split) * 2 + 1] = l;
    }
  }
}

// Joins the key splits of one (sequence, head).
__global__ void latent_decode_merge_kernel(const float* __restrict__ po, const float* __restrict__ ml, const int* __restrict__ ctx_len,
                                           __nv_bfloat16* __restrict__ out, int H, int nsplit, int rank) {
  const long long row = blockIdx.x;
  const float* m = ml + row * nsplit * 2;
  float M = -INFINITY, L = 0.f;
  for (int s = 0; s < nsplit; ++s) M = fmaxf(M, m[2 * s]);
  for (int s = 0; s < nsplit; ++s) L += m[2 * s] == -INFINITY ? 0.f : exp2f(m[2 * s] - M) * m[2 * s + 1];
  const float inv = (L > 0.f && ctx_len[row / H] > 0) ? 1.f / L : 0.f;
  for (int c = threadIdx.x; c < rank; c += blockDim.x) {
    float a = 0.f;
    for (int s = 0; s < nsplit; ++s) a += m[2 * s] == -INFINITY ? 0.f : exp2f(m[2 * s] - M) * po[(row * nsplit + s) * rank + c];
    out[row * rank + c] = __float2bfloat16(a * inv);
  }
}

static int latent_decode_groups(int H) { return H > LD_HEADS ? 2 : 1; }
static int latent_decode_fixed(int panels, int ng) { 
  const int q = LD_HEADS * (panels * 128 + 16), s = 2 * 4 * LD_HEADS * LD_SP * 4;
  return ng * (q > s ? q : s) + 2 * LD_MAX_STAGES * 8 + 1024;
}
static int latent_decode_stages(int panels, int ng) {
  const int s = ((ng == 1 ? 113 * 1024 : 227 * 1024) - latent_decode_fixed(panels, ng)) / (panels * LD_TOK * 128);  // two CTAs per SM / one
  return s < 2 ? 0 : (s > LD_MAX_STAGES ? LD_MAX_STAGES : s);
}

}  // namespace vb

using namespace vb;

// Key splits for S sequences and H heads (0: the sizes are not served). max_keys: most keys a sequence can see.
extern "C" int vb_latent_decode_splits(int S, int H, int rank, int width, int block_size, int max_keys) {
  const int panels = (width + 63) / 64;
  if (rank > 512 || panels > 10 || rank % 8 || width % 8 || rank > width || block_size % 16 || latent_decode_stages(panels, latent_decode_groups(H)) == 0) return 0;
  const int ng = latent_decode_groups(H), groups = S * ((H + ng * LD_HEADS - 1) / (ng * LD_HEADS)), tiles = (max_keys + LD_TOK - 1) / LD_TOK;
  int s = (ng == 1 ? 2 : 1) * num_sms() / groups;
  if (s > tiles / 4) s = tiles / 4;
  return s < 1 ? 1 : (s > 16 ? 16 : s);
}

extern "C" int vb_latent_decode(const VbLatentAttn* a, long long num_blocks, int nsplit, float* part_o, float* part_ml, cudaStream_t stream) {
  const int width = a->du + a->dr, panels = (width + 63) / 64;
  if (a->hq % 8 || a->ldq % 8 || a->page_stride % 8) return -1;
  if ((reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->ku) | reinterpret_cast<uintptr_t>(a->out)) & 15) return -1;
  LatentDecodeParams p{};
  p.box_rows = a->block_size % LD_TOK == 0 ? LD_TOK : 16;
  CUtensorMap tm;
  if (!make_tmap_3d(&tm, a->ku, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, width, a->block_size, num_blocks, a->ku_row, a->page_stride, 64, p.box_rows, 1,
                    CU_TENSOR_MAP_SWIZZLE_128B))
    return -1;
  static int* status = nullptr;
  if (status == nullptr) cudaGetSymbolAddress(reinterpret_cast<void**>(&status), g_latent_decode_status);
  p.q = reinterpret_cast<const __nv_bfloat16*>(a->q); p.ldq = a->ldq; p.hq = a->hq;
  p.block_table = a->block_table; p.max_blocks = a->max_blocks; p.block_size = a->block_size; p.num_blocks = num_blocks;
  p.ctx_len = a->ctx_len; p.sink = reinterpret_cast<const __nv_bfloat16*>(a->sink);
  p.out = reinterpret_cast<__nv_bfloat16*>(a->out); p.part_o = part_o; p.part_ml = part_ml;
  p.H = a->H; p.width = width; p.rank = a->dv; p.panels = panels; p.window = a->window; p.keep = a->window > 0 ? a->keep_first : 0; p.nsplit = nsplit;
  const int ng = latent_decode_groups(a->H);
  p.stages = latent_decode_stages(panels, ng); p.scale_log2 = a->scale * 1.4426950408889634f; p.status = status;
  const int smem = latent_decode_fixed(panels, ng) + p.stages * panels * LD_TOK * 128;
  const dim3 grid(a->B, (a->H + ng * LD_HEADS - 1) / (ng * LD_HEADS), nsplit);
  auto go = [&](auto kern) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<grid, 128 * ng + 32, smem, stream>>>(tm, p);
    return static_cast<int>(cudaGetLastError());
  };
  int rc;
  if (a->dv <= 128 && panels <= 3) rc = ng == 1 ? go(latent_decode_kernel<4, 3, 1>) : go(latent_decode_kernel<4, 3, 2>);
  else if (a->dv <= 256 && panels <= 5) rc = ng == 1 ? go(latent_decode_kernel<8, 5, 1>) : go(latent_decode_kernel<8, 5, 2>);
  else rc = ng == 1 ? go(latent_decode_kernel<16, 10, 1>) : go(latent_decode_kernel<16, 10, 2>);
  if (rc == 0 && nsplit > 1) {
    latent_decode_merge_kernel<<<a->B * a->H, 128, 0, stream>>>(part_o, part_ml, a->ctx_len, p.out, a->H, nsplit, p.rank);
    rc = static_cast<int>(cudaGetLastError());
  }
  return rc;
}

extern "C" int vb_latent_decode_status() {
  int h = 0;
  if (cudaMemcpyFromSymbol(&h, g_latent_decode_status, sizeof(int)) != cudaSuccess) return -1;
  if (h != 0) {
    const int z = 0;
    cudaMemcpyToSymbol(g_latent_decode_status, &z, sizeof(int));
  }
  return h;
}
