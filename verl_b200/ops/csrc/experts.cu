// Routing of mixture-of-experts stacks: sigmoid router with the best `top` experts per token (by corrected scores, inside the
// best groups of experts), and the expert-grouped row
// layout (every expert's rows start at a multiple of 128) filled with copies of the tokens. Two launches, no host
// synchronisation; where a copy sits inside its expert's rows does not matter, so places are handed out by counting.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>

namespace vb {

constexpr int EX_MAX = 1024;   // experts
constexpr int EX_WARPS = 8;

// One warp per token; logits fp32 (columns past E belong to something else). Experts are picked one after the other by the
// largest logit (the sigmoid is monotonic), ties by the smaller index. CHOICE: by the largest sigmoid + correction, among the experts
// of the `keep` best groups (a group's score is the sum of its two largest; ties by the smaller index).
template <int PER_LANE, bool CHOICE, typename T>
__global__ void __launch_bounds__(32 * EX_WARPS)
expert_route_kernel(const float* __restrict__ z, long long ldz, const T* __restrict__ corr, int groups, int keep, int tokens, int E, int k, int renorm,
                    int tokens_per_block, float* __restrict__ score, int* __restrict__ expert, int* __restrict__ rank, int* __restrict__ counts) {
  extern __shared__ float ex_sm[];   // CHOICE: per warp the choice scores [E] and the groups' scores [groups]
  __shared__ int local[EX_MAX];
  for (int e = threadIdx.x; e < E; e += blockDim.x) local[e] = 0;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * tokens_per_block, t1 = min(tokens, t0 + tokens_per_block);
  for (int t = t0 + warp; t < t1; t += EX_WARPS) {
    const float* row = z + static_cast<long long>(t) * ldz;
    float v[PER_LANE];
    unsigned taken = 0;
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
      const bool in = lane + 32 * i < E;
      v[i] = in ? row[lane + 32 * i] : 0.f;
      if (!in) taken |= 1u << i;
    }
    if constexpr (CHOICE) {
      float* sv = ex_sm + warp * (E + groups);
      float* sg = sv + E;
#pragma unroll
      for (int i = 0; i < PER_LANE; ++i)
        if (lane + 32 * i < E) {
          v[i] = sigmoid_f(v[i]) + (corr != nullptr ? to_f(corr[lane + 32 * i]) : 0.f);
          sv[lane + 32 * i] = v[i];
        }
      if (groups > 1) {
        __syncwarp();
        const int size = E / groups;
        for (int g = lane; g < groups; g += 32) {
          float a = -INFINITY, b = -INFINITY;
          for (int e = 0; e < size; ++e) {
            const float x = sv[g * size + e];
            if (x > a) { b = a; a = x; } else b = fmaxf(b, x);
          }
          sg[g] = size > 1 ? a + b : a;
        }
        __syncwarp();
        for (int j = 0; j < keep; ++j) {      // the best group left: marked by +inf
          float best = -INFINITY;
          int bg = 0x7fffffff;
          for (int g = lane; g < groups; g += 32)
            if (sg[g] != INFINITY && (bg == 0x7fffffff || sg[g] > best)) { best = sg[g]; bg = g; }
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int og = __shfl_xor_sync(0xffffffffu, bg, o);
            if (og != 0x7fffffff && (bg == 0x7fffffff || ob > best || (ob == best && og < bg))) { best = ob; bg = og; }
          }
          __syncwarp();
          if (lane == 0 && bg != 0x7fffffff) sg[bg] = INFINITY;
          __syncwarp();
        }
#pragma unroll
        for (int i = 0; i < PER_LANE; ++i)
          if (lane + 32 * i < E && sg[(lane + 32 * i) / size] != INFINITY) taken |= 1u << i;
        __syncwarp();
      }
    }
    float sum = 0.f, my_s = 0.f;
    int my_e = 0;
    for (int j = 0; j < k; ++j) {
      float best = -INFINITY;
      int bi = 0x7fffffff;
#pragma unroll
      for (int i = 0; i < PER_LANE; ++i)
        if (!((taken >> i) & 1u) && (bi == 0x7fffffff || v[i] > best)) { best = v[i]; bi = lane + 32 * i; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (oi != 0x7fffffff && (bi == 0x7fffffff || ob > best || (ob == best && oi < bi))) { best = ob; bi = oi; }
      }
      if ((bi & 31) == lane) taken |= 1u << (bi >> 5);
      const float s = CHOICE ? sigmoid_f(row[bi]) : sigmoid_f(best);
      sum += s;
      if (lane == (j & 31)) { my_s = s; my_e = bi; }
      if ((j & 31) == 31 || j == k - 1) {
        if (lane <= (j & 31)) {
          const long long at = static_cast<long long>(t) * k + (j & ~31) + lane;
          score[at] = my_s;
          expert[at] = my_e;
          rank[at] = atomicAdd(&local[my_e], 1);
        }
      }
    }
    if (renorm)
      for (int j = lane; j < k; j += 32) score[static_cast<long long>(t) * k + j] /= sum + 1e-20f;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x)
    if (local[e] > 0) local[e] = atomicAdd(&counts[e], local[e]);   // the block's first place
  __syncthreads();
  for (long long i = static_cast<long long>(t0) * k + threadIdx.x; i < static_cast<long long>(t1) * k; i += blockDim.x) rank[i] += local[expert[i]];
}

// seg[e] = first row of expert e; copies row h[t] to its place.
template <typename T, int VEC>
__global__ void __launch_bounds__(32 * EX_WARPS)
expert_place_kernel(const T* __restrict__ h, long long ldh, const float* __restrict__ score, const int* __restrict__ expert, const int* __restrict__ rank,
                    const int* __restrict__ counts, long long pairs, int E, int k, int W, T* __restrict__ x, float* __restrict__ row_scale,
                    int* __restrict__ slot, int* __restrict__ tile_expert, int* __restrict__ num_tiles, int max_tiles) {
  __shared__ int seg[EX_MAX + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) {
    const int per = (E + 31) / 32;
    int mine = 0;
    for (int i = 0; i < per; ++i) {
      const int e = lane * per + i;
      if (e < E) mine += (counts[e] + 127) / 128;
    }
    int incl = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += up;
    }
    int at = incl - mine;
    for (int i = 0; i < per; ++i) {
      const int e = lane * per + i;
      if (e < E) {
        seg[e] = at * 128;
        at += (counts[e] + 127) / 128;
      }
    }
    if (lane == 31) seg[E] = at * 128;
  }
  __syncthreads();
  if (blockIdx.x == 0) {
    for (int e = threadIdx.x; e < E; e += blockDim.x)
      for (int i = seg[e] / 128; i < seg[e + 1] / 128 && i < max_tiles; ++i) tile_expert[i] = e;
    if (threadIdx.x == 0) *num_tiles = min(seg[E] / 128, max_tiles);
  }
  for (long long i = blockIdx.x * static_cast<long long>(EX_WARPS) + warp; i < pairs; i += static_cast<long long>(gridDim.x) * EX_WARPS) {
    const int r = seg[expert[i]] + rank[i];
    if (lane == 0) {
      slot[i] = r;
      row_scale[r] = score[i];
    }
    const T* src = h + i / k * ldh;
    T* dst = x + static_cast<long long>(r) * W;
    for (int c = lane * VEC; c < W; c += 32 * VEC) {
      if constexpr (VEC == 8 && sizeof(T) == 2) {
        *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(src + c);
      } else {
        float v[VEC];
        Vec<T, VEC>::load(src + c, v);
        Vec<T, VEC>::store(dst + c, v);
      }
    }
  }
}

}  // namespace vb

using namespace vb;

// counts [E] must be zero; score / expert / rank [T, k].
extern "C" int vb_expert_route(int dtype, const float* z, long long ldz, const void* corr, int groups, int keep, int T, int E, int k, int renorm, float* score,
                               int* expert, int* rank, int* counts, cudaStream_t s) {
  if (T <= 0) return 0;
  if (E < 1 || E > EX_MAX || k < 1 || groups < 1 || E % groups || keep < 1 || keep > groups || k > keep * (E / groups)) return -1;
  const int tpb = T > 148 * 64 ? 32 : EX_WARPS;
  const int blocks = (T + tpb - 1) / tpb;
  const bool choice = corr != nullptr || groups > 1;
  const int smem = choice ? EX_WARPS * (E + groups) * 4 : 0;
  auto go = [&](auto kern, auto* tag) {
    if (smem > 40 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    kern<<<blocks, 32 * EX_WARPS, smem, s>>>(z, ldz, (decltype(tag))corr, groups, keep, T, E, k, renorm, tpb, score, expert, rank, counts);
    return static_cast<int>(cudaGetLastError());
  };
#define EX_ROUTE(C_, T_)                                                                                                                             \
  return E <= 64 ? go(expert_route_kernel<2, C_, T_>, (const T_*)nullptr) : E <= 128 ? go(expert_route_kernel<4, C_, T_>, (const T_*)nullptr)        \
       : E <= 256 ? go(expert_route_kernel<8, C_, T_>, (const T_*)nullptr) : go(expert_route_kernel<32, C_, T_>, (const T_*)nullptr)
  if (!choice) EX_ROUTE(false, float);
  if (dtype == 0) EX_ROUTE(true, float);
  EX_ROUTE(true, __nv_bfloat16);
#undef EX_ROUTE
}

extern "C" int vb_expert_place(int dtype, const void* h, long long ldh, const float* score, const int* expert, const int* rank, const int* counts, int T, int E,
                               int k, int W, void* x, float* row_scale, int* slot, int* tile_expert, int* num_tiles, int max_tiles, cudaStream_t s) {
  if (T <= 0) return 0;
  if (E < 1 || E > EX_MAX) return -1;
  const long long pairs = static_cast<long long>(T) * k, want = (pairs + EX_WARPS - 1) / EX_WARPS;
  const unsigned grid = static_cast<unsigned>(want < 148 * 8 ? want : 148 * 8);
  const bool vec = W % 8 == 0 && ldh % 8 == 0 && ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(x)) & 15) == 0;
  auto go = [&](auto kern, auto* tag) {
    typedef decltype(tag) P;
    kern<<<grid, 32 * EX_WARPS, 0, s>>>((P)h, ldh, score, expert, rank, counts, pairs, E, k, W, (P)x, row_scale, slot, tile_expert, num_tiles, max_tiles);
    return static_cast<int>(cudaGetLastError());
  };
  typedef __nv_bfloat16 bf16;
  if (dtype == 0) return vec ? go(expert_place_kernel<float, 8>, (float*)nullptr) : go(expert_place_kernel<float, 1>, (float*)nullptr);
  return vec ? go(expert_place_kernel<bf16, 8>, (bf16*)nullptr) : go(expert_place_kernel<bf16, 1>, (bf16*)nullptr);
}
