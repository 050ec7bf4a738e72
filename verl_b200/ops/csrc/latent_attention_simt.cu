// Windowed or chunked attention (kept first keys, a sink) over latent or expanded keys, one warp per (query, head), on the fp32 pipeline.
//
// One kernel covers both uses of latent attention: prompts (per-head keys and values expanded from the latents, contiguous
// rows) and decoding (all heads share the latent row as key and value, rows found through the page table), and grouped-query
// attention in both forms (key / value heads shared by groups of query heads, capped scores, pairs of maps over the same values). It serves fp32
// tensors and bf16 sizes outside the tensor-core kernels. Keys are taken 32 at a time: a lane owns a key for the scores, the
// lanes then share the value columns. Compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>

namespace vb {

template <typename T, typename O>
__global__ void __launch_bounds__(128)
latent_attn_simt_kernel(const VbLatentAttn a) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dq = a.du + a.dr;
  float* sq = sm + warp * (dq + a.dv);
  float* so = sq + dq;
  const long long i = blockIdx.x * 4ll + warp;
  if (i >= static_cast<long long>(a.T) * a.H) return;
  const int h = static_cast<int>(i % a.H), maps = a.maps > 1 ? a.maps : 1, vh = a.kv_group > 1 ? h / maps / a.kv_group : h / maps, kh = vh * maps + h % maps;
  const long long t = i / a.H;
  // which sequence, which key rows
  int b = static_cast<int>(t), last;         // index of the query's own key inside its sequence
  long long k_base = 0;
  if (a.cu_q != nullptr) {
    int lo = 0, hi = a.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi) / 2;
      if (a.cu_q[mid + 1] <= t) lo = mid + 1; else hi = mid;
    }
    b = lo;
  }
  if (a.cu_k != nullptr) {
    k_base = a.cu_k[b];
    last = a.cu_k[b + 1] - a.cu_k[b] - 1 - (a.cu_q[b + 1] - 1 - static_cast<int>(t));
  } else {
    last = a.ctx_len[b] - 1;
  }
  O* out = reinterpret_cast<O*>(a.out) + t * a.ldo + static_cast<long long>(h) * a.dv;
  if (last < 0) {
    for (int c = lane; c < a.dv; c += 32) out[c] = from_f<O>(0.f);
    return;
  }
  const T* q = reinterpret_cast<const T*>(a.q) + t * a.ldq + static_cast<long long>(h) * a.hq;
  for (int c = lane; c < dq; c += 32) sq[c] = to_f(q[c]);
  for (int c = lane; c < a.dv; c += 32) so[c] = 0.f;
  __syncwarp();
  const float sink = a.sink != nullptr ? to_f(reinterpret_cast<const T*>(a.sink)[h]) : -INFINITY;
  float m = sink, l = a.sink != nullptr ? 1.f : 0.f;
  const int first = a.window > 0 ? max(0, last - a.window + 1) : a.chunk > 0 ? last / a.chunk * a.chunk : 0, kept = min(a.keep_first, first);
  // the kept keys [0, kept) in front of the window's [first, last]
  for (int j0 = kept > 0 ? 0 : first; j0 <= last; j0 = j0 + 32 < kept || j0 >= first ? j0 + 32 : first) {
    const int j = j0 + lane, end = j0 < first ? kept - 1 : last;
    long long row = 0;
    float s = -INFINITY;
    if (j <= end) {
      if (a.block_table != nullptr)
        row = a.block_table[static_cast<long long>(b) * a.max_blocks + j / a.block_size] * a.page_stride;
      else
        row = k_base + j;
      // page rows: page_stride counts elements of the latent tensor; contiguous rows are scaled by the row strides
      const T *ku, *kr;
      if (a.block_table != nullptr) {
        row += static_cast<long long>(j % a.block_size) * a.ku_row;
        ku = reinterpret_cast<const T*>(a.ku) + row + static_cast<long long>(kh) * a.ku_head;
        kr = reinterpret_cast<const T*>(a.kr) + row;
      } else {
        ku = reinterpret_cast<const T*>(a.ku) + row * a.ku_row + static_cast<long long>(kh) * a.ku_head;
        kr = reinterpret_cast<const T*>(a.kr) + row * a.kr_row;
      }
      float acc = 0.f;
      for (int c = 0; c < a.du; ++c) acc = fmaf(sq[c], to_f(ku[c]), acc);
      for (int c = 0; c < a.dr; ++c) acc = fmaf(sq[a.du + c], to_f(kr[c]), acc);
      s = acc * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float alpha = expf(m - m_new);
    const float p = j <= end ? expf(s - m_new) : 0.f;
    l = l * alpha + warp_sum(p);
    m = m_new;
    for (int c = lane; c < a.dv; c += 32) so[c] *= alpha;
    const int n = min(32, end - j0 + 1);
    for (int jj = 0; jj < n; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const long long rj = __shfl_sync(0xffffffffu, row, jj);
      const T* v = reinterpret_cast<const T*>(a.v) + (a.block_table != nullptr ? rj : rj * a.v_row) + static_cast<long long>(vh) * a.v_head;
      for (int c = lane; c < a.dv; c += 32) so[c] = fmaf(pj, to_f(v[c]), so[c]);
    }
  }
  const float f = (a.gate != nullptr ? sigmoid_f(a.gate[t * a.ldg + h]) : 1.f) / l;
  for (int c = lane; c < a.dv; c += 32) out[c] = from_f<O>(so[c] * f);
}

}  // namespace vb

using namespace vb;

extern "C" int vb_latent_attn_simt(int dtype, const VbLatentAttn* a, int out_f32, cudaStream_t s) {
  if (a->T <= 0) return 0;
  const int smem = 4 * (a->du + a->dr + a->dv) * 4;
  if (smem > 200 * 1024) return -2;
  const long long warps = static_cast<long long>(a->T) * a->H;
  const unsigned grid = static_cast<unsigned>((warps + 3) / 4);
  auto go = [&](auto kern) {
    if (smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    kern<<<grid, 128, smem, s>>>(*a);
    return static_cast<int>(cudaGetLastError());
  };
  if (dtype == 0) return go(latent_attn_simt_kernel<float, float>);
  return out_f32 ? go(latent_attn_simt_kernel<__nv_bfloat16, float>) : go(latent_attn_simt_kernel<__nv_bfloat16, __nv_bfloat16>);
}
