// GEMM on the fp32 pipeline: D = A B^T with fp32 products and sums, for fp32 operands (exact 32-bit inference) and for
// bf16 operands whose sizes or strides the TMA kernels do not serve (rows that are not a multiple of 16 bytes).
// 64 x 64 tile per CTA, 4 x 4 outputs per thread, optional batch over gridDim.z. Compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

namespace vb {

constexpr int SG_T = 64, SG_K = 16;

template <typename T>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ A, const T* __restrict__ B, int M, int N, int K, long long lda, long long ldb, int b_mn,
                 long long sa, long long sb, long long sd, VbEpiArgs e, const int* __restrict__ tile_expert, const int* __restrict__ num_tiles) {
  if (tile_expert != nullptr) {            // rows grouped by expert, 128 to a tile
    const int tile = blockIdx.y * SG_T / 128;
    if (tile >= *num_tiles) return;
    B += static_cast<long long>(tile_expert[tile]) * N * K;
  }
  __shared__ float As[SG_K][SG_T + 4], Bs[SG_K][SG_T + 4];
  A += blockIdx.z * sa;
  B += blockIdx.z * sb;
  const int m0 = blockIdx.y * SG_T, n0 = blockIdx.x * SG_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += SG_K) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int i = threadIdx.x + u * 256;
      const int kk = i & 15, r = i >> 4;
      As[kk][r] = (m0 + r < M && k0 + kk < K) ? to_f(A[(m0 + r) * lda + k0 + kk]) : 0.f;
      if (!b_mn) {
        Bs[kk][r] = (n0 + r < N && k0 + kk < K) ? to_f(B[(n0 + r) * ldb + k0 + kk]) : 0.f;
      } else {
        const int rn = i & 63, kb = i >> 6;
        Bs[kb][rn] = (n0 + rn < N && k0 + kb < K) ? to_f(B[(k0 + kb) * ldb + n0 + rn]) : 0.f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < SG_K; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = As[kk][ty * 4 + i]; b[i] = Bs[kk][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
  const float alpha = (e.mode == VB_EPI_RESID && e.D != nullptr) ? to_f(*reinterpret_cast<const T*>(e.alpha)) : 0.f;
  const float palpha = (e.mode == VB_EPI_RESID && e.pw != nullptr) ? to_f(*reinterpret_cast<const T*>(e.palpha)) : 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = acc[i][j];
      T* D = reinterpret_cast<T*>(e.D) + blockIdx.z * sd;
      switch (e.mode) {
        case VB_EPI_STORE:
          if (e.gate != nullptr) v *= sigmoid_f(e.gate[m * e.ldg + blockIdx.z]);
          D[m * e.ldd + n] = from_f<T>(v); break;
        case VB_EPI_STORE_F32: (reinterpret_cast<float*>(e.D) + blockIdx.z * sd)[m * e.ldd + n] = v; break;
        case VB_EPI_SOFTCAP: D[m * e.ldd + n] = from_f<T>(e.cap * tanhf(v / e.cap)); break;
        case VB_EPI_GELU: D[m * e.ldd + n] = from_f<T>(gelu_erf(v)); break;
        case VB_EPI_BIAS: D[m * e.ldd + n] = from_f<T>(v + to_f(reinterpret_cast<const T*>(e.nb)[n])); break;
        case VB_EPI_SILU: D[m * e.ldd + n] = from_f<T>(n < e.n0 ? v * sigmoid_f(v) : v); break;
        case VB_EPI_BIAS_RELU2: {
          const float z = fmaxf(v + to_f(reinterpret_cast<const T*>(e.nb)[n]), 0.f);
          D[m * e.ldd + n] = from_f<T>(z * z); break;
        }
        case VB_EPI_TANH: D[m * e.ldd + n] = from_f<T>(n < e.n0 ? v : tanhf(v)); break;
        case VB_EPI_SPLIT:
          if (n < e.n0) D[m * e.ldd + n] = from_f<T>(v);
          else e.D2[m * e.ldd2 + n - e.n0] = v;
          break;
        default: {
          if (e.pw != nullptr) v = tanhf(palpha * v) * to_f(reinterpret_cast<const T*>(e.pw)[n]) + to_f(reinterpret_cast<const T*>(e.pb)[n]);
          else if (e.pb != nullptr) v += to_f(reinterpret_cast<const T*>(e.pb)[n]);
          const float x = e.X[m * e.ldx + n] + v;
          e.X[m * e.ldx + n] = x;
          if (e.D != nullptr)
            D[m * e.ldd + n] = from_f<T>(tanhf(alpha * x) * to_f(reinterpret_cast<const T*>(e.nw)[n]) + to_f(reinterpret_cast<const T*>(e.nb)[n]));
        }
      }
    }
  }
}

}  // namespace vb

using namespace vb;

static int simt_launch(int dtype, const void* A, const void* B, int M, int N, int K, long long lda, long long ldb, int b_mn, int batch,
                       long long sa, long long sb, long long sd, const VbEpiArgs* e, const int* tile_expert, const int* num_tiles, cudaStream_t s) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  dim3 grid((N + SG_T - 1) / SG_T, (M + SG_T - 1) / SG_T, batch);
  if (grid.y > 65535 || grid.z > 65535) return -1;
  if (dtype == 0)
    gemm_simt_kernel<float><<<grid, 256, 0, s>>>((const float*)A, (const float*)B, M, N, K, lda, ldb, b_mn, sa, sb, sd, *e, tile_expert, num_tiles);
  else
    gemm_simt_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>((const __nv_bfloat16*)A, (const __nv_bfloat16*)B, M, N, K, lda, ldb, b_mn, sa, sb, sd, *e, tile_expert, num_tiles);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_gemm_simt(int dtype, const void* A, const void* B, int M, int N, int K, long long lda, long long ldb, int b_mn, int batch,
                            long long sa, long long sb, long long sd, const VbEpiArgs* e, cudaStream_t s) {
  return simt_launch(dtype, A, B, M, N, K, lda, ldb, b_mn, batch, sa, sb, sd, e, nullptr, nullptr, s);
}

extern "C" int vb_gemm_simt_grouped(int dtype, const void* A, const void* B, int M, int N, int K, long long lda, const int* tile_expert, const int* num_tiles,
                                    const VbEpiArgs* e, cudaStream_t s) {
  return simt_launch(dtype, A, B, M, N, K, lda, K, 0, 1, 0, 0, 0, e, tile_expert, num_tiles, s);
}
