// Mixer-stack kernels around the matrix products: scaled embedding with the first norm, Dynamic Tanh, pairwise rotation,
// the latent-attention preparation (two RMS norms, rotation of the shared key part, append to the paged cache), and the
// mLSTM recurrence (single step for decoding, token-by-token scan, output norm and gate).
// Statistics, angles, gates and recurrent state are fp32; compiled without fast math.
#include "mixers.h"
#include "mixer_common.cuh"

#include <math.h>

namespace vb {

typedef __nv_bfloat16 bf16;

// --------------------------------------------------------------------------------------------- embedding + Dynamic Tanh
template <typename T, int VEC>
__global__ void embed_dyt_kernel(const long long* __restrict__ ids, const T* __restrict__ w, float scale, float* __restrict__ x,
                                 T* __restrict__ h, const T* __restrict__ alpha, const T* __restrict__ nw, const T* __restrict__ nb,
                                 const T* __restrict__ ealpha, const T* __restrict__ ew, const T* __restrict__ eb, int W, int V) {
  const long long t = blockIdx.x;
  const long long id = ids == nullptr ? 0 : ids[t];
  const bool ok = ids == nullptr || (id >= 0 && id < V);
  const float a = h != nullptr ? to_f(*alpha) : 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC], g[VEC], b[VEC];
    if (ids == nullptr) {
      Vec<float, VEC>::load(x + t * W + c, v);
    } else {
      if (ok) Vec<T, VEC>::load(w + id * W + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = ok ? v[i] * scale : 0.f;
      if (ew != nullptr) {               // the embedding passes a norm of its own
        const float ea = to_f(*ealpha);
        Vec<T, VEC>::load(ew + c, g);
        Vec<T, VEC>::load(eb + c, b);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = tanhf(ea * v[i]) * g[i] + b[i];
      }
      Vec<float, VEC>::store(x + t * W + c, v);
    }
    if (h != nullptr) {
      Vec<T, VEC>::load(nw + c, g);
      Vec<T, VEC>::load(nb + c, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = tanhf(a * v[i]) * g[i] + b[i];
      Vec<T, VEC>::store(h + t * W + c, v);
    }
  }
}

template <typename T>
static int embed_dyt(const long long* ids, const void* w, float scale, float* x, void* h, const void* alpha, const void* nw, const void* nb,
                     const void* ea, const void* ew, const void* eb, int T_, int W, int V, cudaStream_t s) {
  const int thr = W >= 1024 ? 256 : 128;
  if (W % 8 == 0)
    embed_dyt_kernel<T, 8><<<T_, thr, 0, s>>>(ids, (const T*)w, scale, x, (T*)h, (const T*)alpha, (const T*)nw, (const T*)nb, (const T*)ea, (const T*)ew,
                                               (const T*)eb, W, V);
  else
    embed_dyt_kernel<T, 1><<<T_, thr, 0, s>>>(ids, (const T*)w, scale, x, (T*)h, (const T*)alpha, (const T*)nw, (const T*)nb, (const T*)ea, (const T*)ew,
                                               (const T*)eb, W, V);
  return static_cast<int>(cudaGetLastError());
}

// --------------------------------------------------------------------------------------------- pairwise rotation
// Dimensions off + 2i and off + 2i + 1 of every head form a pair, i < dims / 2; cos / sin tables [max_pos, dims / 2].
template <typename T>
__global__ void rope_pairs_kernel(T* __restrict__ x, const int* __restrict__ pos, const float* __restrict__ cs, const float* __restrict__ sn,
                                  int heads, long long ld, int hstride, int off, int half, int max_pos, long long total) {
  const long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x;
  if (i >= total) return;
  const int p = static_cast<int>(i % half);
  const long long th = i / half;
  const int hd = static_cast<int>(th % heads);
  const long long t = th / heads;
  const int at = min(max(pos[t], 0), max_pos - 1);
  T* e = x + t * ld + static_cast<long long>(hd) * hstride + off + 2 * p;
  const float u = to_f(e[0]), v = to_f(e[1]);
  const float c = cs[static_cast<long long>(at) * half + p], s = sn[static_cast<long long>(at) * half + p];
  e[0] = from_f<T>(u * c - v * s);
  e[1] = from_f<T>(v * c + u * s);
}

// Out of place, between rows of different layout; dimensions behind the rotated ones are copied.
template <typename T>
__global__ void rope_copy_kernel(const T* __restrict__ a, long long lda, int a_head, int a_off, T* __restrict__ out, long long ldo, int o_head, int o_off,
                                 const int* __restrict__ pos, const float* __restrict__ cs, const float* __restrict__ sn, int heads, int rot, int half,
                                 int max_pos, long long total) {
  const long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x;
  if (i >= total) return;
  const int c = static_cast<int>(i % rot);
  const long long th = i / rot, t = th / heads;
  const int hd = static_cast<int>(th % heads);
  const T* src = a + t * lda + static_cast<long long>(hd) * a_head + a_off;
  float o = to_f(src[c]);
  if (c < 2 * half) {
    const long long at = static_cast<long long>(min(max(pos[t], 0), max_pos - 1)) * half + (c >> 1);
    const float w = to_f(src[c ^ 1]);
    o = (c & 1) ? o * cs[at] + w * sn[at] : o * cs[at] - w * sn[at];
  }
  out[t * ldo + static_cast<long long>(hd) * o_head + o_off + c] = from_f<T>(o);
}

// --------------------------------------------------------------------------------------------- latent preparation
// Row p[t] = [query latent (q_rank) | key/value latent (kv_rank) | shared key part (rot)]: RMS norms of the two latents,
// rotation of the key part; the latent row (kv_rank + rot) goes to `lat` and / or to its place in the paged cache.
template <typename T, int VEC>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const T* __restrict__ p, long long ldp, const T* __restrict__ qn, const T* __restrict__ kn, float eps,
                   const int* __restrict__ pos, const float* __restrict__ cs, const float* __restrict__ sn, int dims, int max_pos,
                   T* __restrict__ cq, T* __restrict__ lat, long long ldl, T* __restrict__ pages, long long page_stride, int block_size,
                   long long num_slots, const long long* __restrict__ slot, int q_rank, int kv_rank, int rot) {
  __shared__ float red[33];
  const long long t = blockIdx.x;
  const T* row = p + t * ldp;
  const int width = kv_rank + rot;
  T* page = nullptr;
  if (pages != nullptr) {
    const long long sl = slot[t];
    if (sl >= 0 && sl < num_slots) page = pages + (sl / block_size) * page_stride + (sl % block_size) * width;
  }
  T* lrow = lat != nullptr ? lat + t * ldl : nullptr;
  float sq = 0.f, sk = 0.f, v[VEC], g[VEC];
  for (int c = threadIdx.x * VEC; c < q_rank; c += blockDim.x * VEC) {
    Vec<T, VEC>::load(row + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) sq += v[i] * v[i];
  }
  for (int c = threadIdx.x * VEC; c < kv_rank; c += blockDim.x * VEC) {
    Vec<T, VEC>::load(row + q_rank + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) sk += v[i] * v[i];
  }
  sq = block_sum(sq, red);
  sk = block_sum(sk, red);
  const float rq = 1.f / sqrtf(sq / q_rank + eps), rk = 1.f / sqrtf(sk / kv_rank + eps);
  for (int c = threadIdx.x * VEC; c < q_rank; c += blockDim.x * VEC) {
    Vec<T, VEC>::load(row + c, v);
    Vec<T, VEC>::load(qn + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * rq * g[i];
    Vec<T, VEC>::store(cq + t * q_rank + c, v);
  }
  for (int c = threadIdx.x * VEC; c < kv_rank; c += blockDim.x * VEC) {
    Vec<T, VEC>::load(row + q_rank + c, v);
    Vec<T, VEC>::load(kn + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * rk * g[i];
    if (lrow != nullptr) Vec<T, VEC>::store(lrow + c, v);
    if (page != nullptr) Vec<T, VEC>::store(page + c, v);
  }
  const T* kr = row + q_rank + kv_rank;
  const int at = min(max(pos[t], 0), max_pos - 1), half = dims / 2;
  for (int c = threadIdx.x; c < rot; c += blockDim.x) {
    float o = to_f(kr[c]);
    if (c < 2 * half) {
      const float cc = cs[static_cast<long long>(at) * half + (c >> 1)], ss = sn[static_cast<long long>(at) * half + (c >> 1)];
      const float w = to_f(kr[c ^ 1]);
      o = (c & 1) ? o * cc + w * ss : o * cc - w * ss;
    }
    if (lrow != nullptr) lrow[kv_rank + c] = from_f<T>(o);
    if (page != nullptr) page[kv_rank + c] = from_f<T>(o);
  }
}

// The same without a query latent: one warp per token, the row in registers (kv_rank <= 1024, sizes multiples of 8).
template <int ITEMS>
__global__ void __launch_bounds__(256)
latent_row_kernel(const bf16* __restrict__ p, long long ldp, const bf16* __restrict__ kn, float eps, const int* __restrict__ pos, const float* __restrict__ cs,
                  const float* __restrict__ sn, int half, int max_pos, bf16* __restrict__ lat, long long ldl, bf16* __restrict__ pages, long long page_stride,
                  int block_size, long long num_slots, const long long* __restrict__ slot, int T, int kv_rank, int rot) {
  const long long t = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= T) return;
  const bf16* row = p + t * ldp;
  float v[ITEMS][8], r8[8], g[8], sum = 0.f;
  const int rc = lane * 8;                                   // this lane's part of the shared key part
  if (rc < rot) Vec<bf16, 8>::load(row + kv_rank + rc, r8);
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * 32 + lane) * 8;
    if (c >= kv_rank) continue;
    Vec<bf16, 8>::load(row + c, v[i]);
#pragma unroll
    for (int k = 0; k < 8; ++k) sum += v[i][k] * v[i][k];
  }
  bf16 *d0 = lat != nullptr ? lat + t * ldl : nullptr, *d1 = nullptr;
  if (pages != nullptr) {
    const long long sl = slot[t];
    if (sl >= 0 && sl < num_slots) {
      const unsigned blk = static_cast<unsigned>(sl) / static_cast<unsigned>(block_size);
      d1 = pages + blk * page_stride + static_cast<long long>(static_cast<unsigned>(sl) - blk * block_size) * (kv_rank + rot);
    }
  }
  const float r = 1.f / sqrtf(warp_sum(sum) / kv_rank + eps);
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * 32 + lane) * 8;
    if (c >= kv_rank) continue;
    Vec<bf16, 8>::load(kn + c, g);
#pragma unroll
    for (int k = 0; k < 8; ++k) v[i][k] *= r * g[k];
    if (d0 != nullptr) Vec<bf16, 8>::store(d0 + c, v[i]);
    if (d1 != nullptr) Vec<bf16, 8>::store(d1 + c, v[i]);
  }
  if (rc < rot) {
    const long long tab = static_cast<long long>(min(max(pos[t], 0), max_pos - 1)) * half;
#pragma unroll
    for (int k = 0; k < 8; k += 2)
      if (rc + k < 2 * half) {
        const float c = cs[tab + ((rc + k) >> 1)], s = sn[tab + ((rc + k) >> 1)], x = r8[k], y = r8[k + 1];
        r8[k] = x * c - y * s;
        r8[k + 1] = y * c + x * s;
      }
    if (d0 != nullptr) Vec<bf16, 8>::store(d0 + kv_rank + rc, r8);
    if (d1 != nullptr) Vec<bf16, 8>::store(d1 + kv_rank + rc, r8);
  }
}

// Rows of the paged cache laid out contiguously: sequence b contributes the tokens k_start[b] .. of its block table.
template <typename T>
__global__ void gather_pages_kernel(const T* __restrict__ pages, long long page_stride, int block_size, const int* __restrict__ bt,
                                    int max_blocks, const int* __restrict__ cu_k, const int* __restrict__ k_start, int B, int width,
                                    T* __restrict__ out) {
  const int r = blockIdx.x;
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi) / 2;
    if (cu_k[mid + 1] <= r) lo = mid + 1; else hi = mid;
  }
  const int tok = k_start[lo] + r - cu_k[lo];
  const int blk = min(tok / block_size, max_blocks - 1);
  const T* src = pages + static_cast<long long>(bt[static_cast<long long>(lo) * max_blocks + blk]) * page_stride + static_cast<long long>(tok % block_size) * width;
  for (int c = threadIdx.x; c < width; c += blockDim.x) out[static_cast<long long>(r) * width + c] = src[c];
}

// --------------------------------------------------------------------------------------------- mLSTM
struct Gates { float i, f; };
template <typename T>
__device__ __forceinline__ Gates mlstm_gates(const float* __restrict__ gates, long long ldg, const T* ib, const T* fb, float cap, long long t, int h, int H) {
  Gates g;
  g.i = cap * tanhf((gates[t * ldg + h] + to_f(ib[h])) / cap);
  g.f = log_sigmoid(cap * tanhf((gates[t * ldg + H + h] + to_f(fb[h])) / cap));
  return g;
}

// Per (slot, head) state: S [d, e], then n [d], then m, all heads of a layer packed as H x (d * e + d + 1) floats... laid out as
// S of all heads, n of all heads, m of all heads.
__device__ __forceinline__ float* st_S(float* s, int h, int d, int e) { return s + static_cast<long long>(h) * d * e; }
__device__ __forceinline__ float* st_n(float* s, int h, int H, int d, int e) { return s + static_cast<long long>(H) * d * e + h * d; }
__device__ __forceinline__ float* st_m(float* s, int h, int H, int d, int e) { return s + static_cast<long long>(H) * d * e + H * d + h; }

// One decode step of one (slot, head): state update, read-out, per-head RMS norm, weight and output gate.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
mlstm_decode_kernel(const T* __restrict__ qkvg, long long ldp, const float* __restrict__ gates, long long ldg, const T* __restrict__ ib,
                    const T* __restrict__ fb, float cap, float* __restrict__ state, long long slot_stride, const uint8_t* __restrict__ active,
                    const T* __restrict__ norm, float eps, T* __restrict__ out, long long ldo, int H, int d, int e) {
  extern __shared__ float sm[];
  __shared__ float red[33];
  const int h = blockIdx.x, tid = threadIdx.x;
  const long long t = blockIdx.y;
  T* orow = out + t * ldo + static_cast<long long>(h) * e;
  if (active != nullptr && !active[t]) {
    for (int c = tid; c < e; c += blockDim.x) orow[c] = from_f<T>(0.f);
    return;
  }
  float* sq = sm;            // [d]
  float* sk = sq + d;        // [d]
  float* so = sk + d;        // [row groups][e]
  float* st = state + t * slot_stride;
  float* S = st_S(st, h, d, e);
  float* n = st_n(st, h, H, d, e);
  float* mp = st_m(st, h, H, d, e);
  const T* row = qkvg + t * ldp;
  const float qs = 1.f / sqrtf(static_cast<float>(d));
  const Gates g = mlstm_gates(gates, ldg, ib, fb, cap, t, h, H);
  const float m_old = *mp;
  const float m_new = fmaxf(g.f + m_old, g.i);
  const float keep = expf(g.f + m_old - m_new), add = expf(g.i - m_new);
  float nq = 0.f;
  for (int r = tid; r < d; r += blockDim.x) {
    const float q = to_f(row[h * d + r]) * qs, k = to_f(row[(H + h) * d + r]);
    sq[r] = q;
    sk[r] = add * k;
    const float nn = keep * n[r] + add * k;
    n[r] = nn;
    nq += nn * q;
  }
  nq = block_sum(nq, red);   // also orders the shared q / k writes before their use
  const float den = fmaxf(fabsf(nq), expf(-m_new)) + 1e-6f;
  const int cg = (e + VEC - 1) / VEC;             // column groups
  const int tpc = min(cg, static_cast<int>(blockDim.x));
  const int rgs = blockDim.x / tpc;
  const int rg = tid / tpc, ct = tid % tpc;
  const T* vrow = row + 2 * H * d + static_cast<long long>(h) * e;
  if (rg < rgs) {
    for (int c = ct; c < cg; c += tpc) {
      float v[VEC], o[VEC] = {};
      Vec<T, VEC>::load(vrow + c * VEC, v);
      float* Sc = S + c * VEC;
      int r = rg;
      for (; r + 3 * rgs < d; r += 4 * rgs) {
        float s4[4][VEC];
#pragma unroll
        for (int u = 0; u < 4; ++u) Vec<float, VEC>::load(Sc + static_cast<long long>(r + u * rgs) * e, s4[u]);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float k = sk[r + u * rgs], q = sq[r + u * rgs];
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            s4[u][i] = keep * s4[u][i] + k * v[i];
            o[i] += s4[u][i] * q;
          }
          Vec<float, VEC>::store(Sc + static_cast<long long>(r + u * rgs) * e, s4[u]);
        }
      }
      for (; r < d; r += rgs) {
        float s1[VEC];
        Vec<float, VEC>::load(Sc + static_cast<long long>(r) * e, s1);
        const float k = sk[r], q = sq[r];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          s1[i] = keep * s1[i] + k * v[i];
          o[i] += s1[i] * q;
        }
        Vec<float, VEC>::store(Sc + static_cast<long long>(r) * e, s1);
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) so[rg * e + c * VEC + i] = o[i];
    }
  }
  if (tid == 0) *mp = m_new;
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < e; c += blockDim.x) {
    float o = 0.f;
    for (int u = 0; u < rgs; ++u) o += so[u * e + c];
    o /= den;
    so[c] = o;
    ss += o * o;
  }
  ss = block_sum(ss, red);
  const float rs = 1.f / sqrtf(ss / e + eps);
  const T* grow = row + 2 * H * d + static_cast<long long>(H) * e + static_cast<long long>(h) * e;
  for (int c = tid; c < e; c += blockDim.x)
    orow[c] = from_f<T>(so[c] * rs * to_f(norm[h * e + c]) * sigmoid_f(to_f(grow[c])));
}

// Token-by-token scan of a portion: one CTA = one (sequence, head, 32 columns of e); the state columns live in shared memory.
constexpr int SCAN_COLS = 32, SCAN_ROWS = 8;  // 8 row groups x 32 columns = 256 threads
template <typename T>
__global__ void __launch_bounds__(SCAN_COLS * SCAN_ROWS)
mlstm_scan_kernel(const T* __restrict__ qkvg, long long ldp, const float* __restrict__ gates, long long ldg, const T* __restrict__ ib,
                  const T* __restrict__ fb, float cap, float* __restrict__ state, long long slot_stride, const int* __restrict__ slots,
                  const int* __restrict__ fresh, const int* __restrict__ cu, float* __restrict__ o, int H, int d, int e) {
  extern __shared__ float sm[];
  __shared__ float part[SCAN_ROWS][SCAN_COLS];
  __shared__ float nqs[SCAN_ROWS];
  float* S = sm;                       // [d][32]
  float* sq = S + d * SCAN_COLS;       // [d]
  float* sk = sq + d;                  // [d]
  float* n = sk + d;                   // [d]
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * SCAN_COLS;
  const int c = threadIdx.x, rg = threadIdx.y, tid = rg * SCAN_COLS + c;
  const bool c_ok = c0 + c < e;
  const bool have = slots != nullptr && slots[b] >= 0;
  float* st = have ? state + static_cast<long long>(slots[b]) * slot_stride : nullptr;
  const bool zero = !have || fresh == nullptr || fresh[b] != 0;
  float m = zero ? 0.f : *st_m(st, h, H, d, e);
  for (int r = rg; r < d; r += SCAN_ROWS) S[r * SCAN_COLS + c] = (zero || !c_ok) ? 0.f : st_S(st, h, d, e)[static_cast<long long>(r) * e + c0 + c];
  for (int r = tid; r < d; r += SCAN_COLS * SCAN_ROWS) n[r] = zero ? 0.f : st_n(st, h, H, d, e)[r];
  const float qs = 1.f / sqrtf(static_cast<float>(d));
  __syncthreads();
  for (long long t = cu[b]; t < cu[b + 1]; ++t) {
    const T* row = qkvg + t * ldp;
    const Gates g = mlstm_gates(gates, ldg, ib, fb, cap, t, h, H);
    const float m_new = fmaxf(g.f + m, g.i);
    const float keep = expf(g.f + m - m_new), add = expf(g.i - m_new);
    m = m_new;
    float nq = 0.f;
    for (int r = tid; r < d; r += SCAN_COLS * SCAN_ROWS) {
      const float q = to_f(row[h * d + r]) * qs, k = add * to_f(row[(H + h) * d + r]);
      sq[r] = q;
      sk[r] = k;
      n[r] = keep * n[r] + k;
      nq += n[r] * q;
    }
    nq = warp_sum(nq);
    if (c == 0) nqs[rg] = nq;
    __syncthreads();
    const float v = c_ok ? to_f(row[2 * H * d + h * e + c0 + c]) : 0.f;
    float acc = 0.f;
    for (int r = rg; r < d; r += SCAN_ROWS) {
      const float s = keep * S[r * SCAN_COLS + c] + sk[r] * v;
      S[r * SCAN_COLS + c] = s;
      acc += s * sq[r];
    }
    part[rg][c] = acc;
    __syncthreads();
    if (rg == 0 && c_ok) {
      float a = 0.f, z = 0.f;
#pragma unroll
      for (int u = 0; u < SCAN_ROWS; ++u) { a += part[u][c]; z += nqs[u]; }
      o[(t * H + h) * e + c0 + c] = a / (fmaxf(fabsf(z), expf(-m)) + 1e-6f);
    }
    __syncthreads();
  }
  if (have) {
    for (int r = rg; r < d; r += SCAN_ROWS)
      if (c_ok) st_S(st, h, d, e)[static_cast<long long>(r) * e + c0 + c] = S[r * SCAN_COLS + c];
    // every column block of the head read n and m before any of them may overwrite them only if the values agree: they
    // are written back by a separate launch (mlstm_scan_tail_kernel)
  }
}

// n and m after a portion (the scan's column blocks all start from the same stored n and m, so they must not be replaced
// while a block may still read them).
template <typename T>
__global__ void mlstm_scan_tail_kernel(const T* __restrict__ qkvg, long long ldp, const float* __restrict__ gates, long long ldg,
                                       const T* __restrict__ ib, const T* __restrict__ fb, float cap, float* __restrict__ state,
                                       long long slot_stride, const int* __restrict__ slots, const int* __restrict__ fresh,
                                       const int* __restrict__ cu, int H, int d, int e) {
  const int b = blockIdx.y, h = blockIdx.x;
  if (slots == nullptr || slots[b] < 0) return;
  float* st = state + static_cast<long long>(slots[b]) * slot_stride;
  const bool zero = fresh == nullptr || fresh[b] != 0;
  float* n = st_n(st, h, H, d, e);
  const float m0 = zero ? 0.f : *st_m(st, h, H, d, e);
  float m = m0;
  for (int r0 = 0; r0 < d; r0 += blockDim.x) {
    const int r = r0 + threadIdx.x;
    float nn = (zero || r >= d) ? 0.f : n[r];
    m = m0;
    for (long long t = cu[b]; t < cu[b + 1]; ++t) {
      const Gates g = mlstm_gates(gates, ldg, ib, fb, cap, t, h, H);
      const float m_new = fmaxf(g.f + m, g.i);
      const float k = r < d ? expf(g.i - m_new) * to_f(qkvg[t * ldp + (H + h) * d + r]) : 0.f;
      nn = expf(g.f + m - m_new) * nn + k;
      m = m_new;
    }
    if (r < d) n[r] = nn;
  }
  __syncthreads();
  if (threadIdx.x == 0) *st_m(st, h, H, d, e) = m;
}

// Per-head RMS norm, weight, output gate: out = o / rms(o) * norm * sigmoid(g). One warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
mlstm_out_kernel(const float* __restrict__ o, const T* __restrict__ g, long long ldg, const T* __restrict__ norm, float eps,
                 T* __restrict__ out, long long ldo, long long total, int H, int e) {
  const long long i = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (i >= total) return;
  const int lane = threadIdx.x & 31, h = static_cast<int>(i % H);
  const long long t = i / H;
  const float* src = o + i * e;
  float ss = 0.f;
  for (int c = lane; c < e; c += 32) ss += src[c] * src[c];
  const float rs = 1.f / sqrtf(warp_sum(ss) / e + eps);
  for (int c = lane; c < e; c += 32)
    out[t * ldo + h * e + c] = from_f<T>(src[c] * rs * to_f(norm[h * e + c]) * sigmoid_f(to_f(g[t * ldg + h * e + c])));
}

constexpr int MAX_SMEM = 232448 - 2048;
template <typename K>
static int allow_smem(K kern, int bytes) {
  if (bytes > MAX_SMEM) return -2;
  if (bytes > 48 * 1024) return static_cast<int>(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
  return 0;
}

template <typename T, int VEC>
static int mlstm_decode(const void* qkvg, long long ldp, const float* gates, long long ldg, const void* ib, const void* fb, float cap,
                        float* state, long long slot_stride, const uint8_t* active, const void* norm, float eps, void* out, long long ldo,
                        int S, int H, int d, int e, cudaStream_t s) {
  const int cg = (e + VEC - 1) / VEC, tpc = cg < 256 ? cg : 256, rgs = 256 / tpc;
  const int smem = (2 * d + rgs * e) * 4;
  const int rc = allow_smem(mlstm_decode_kernel<T, VEC>, smem);
  if (rc != 0) return rc;
  mlstm_decode_kernel<T, VEC><<<dim3(H, S), 256, smem, s>>>((const T*)qkvg, ldp, gates, ldg, (const T*)ib, (const T*)fb, cap, state,
                                                             slot_stride, active, (const T*)norm, eps, (T*)out, ldo, H, d, e);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int mlstm_scan(const void* qkvg, long long ldp, const float* gates, long long ldg, const void* ib, const void* fb, float cap,
                      float* state, long long slot_stride, const int* slots, const int* fresh, const int* cu, int B, float* o, int H, int d,
                      int e, cudaStream_t s) {
  const int smem = (d * SCAN_COLS + 3 * d) * 4;
  const int rc = allow_smem(mlstm_scan_kernel<T>, smem);
  if (rc != 0) return rc;
  mlstm_scan_kernel<T><<<dim3((e + SCAN_COLS - 1) / SCAN_COLS, H, B), dim3(SCAN_COLS, SCAN_ROWS), smem, s>>>(
      (const T*)qkvg, ldp, gates, ldg, (const T*)ib, (const T*)fb, cap, state, slot_stride, slots, fresh, cu, o, H, d, e);
  if (slots != nullptr)
    mlstm_scan_tail_kernel<T><<<dim3(H, B), 128, 0, s>>>((const T*)qkvg, ldp, gates, ldg, (const T*)ib, (const T*)fb, cap, state, slot_stride,
                                                         slots, fresh, cu, H, d, e);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace vb

using namespace vb;

extern "C" int vb_embed_dyt(int dtype, const long long* ids, const void* w, float scale, float* x, void* h, const void* alpha, const void* nw,
                            const void* nb, int T, int W, int V, cudaStream_t s) {
  if (T <= 0) return 0;
  return dtype == 0 ? embed_dyt<float>(ids, w, scale, x, h, alpha, nw, nb, nullptr, nullptr, nullptr, T, W, V, s)
                    : embed_dyt<bf16>(ids, w, scale, x, h, alpha, nw, nb, nullptr, nullptr, nullptr, T, W, V, s);
}
extern "C" int vb_embed_dyt2(int dtype, const long long* ids, const void* w, float* x, void* h, const void* ealpha, const void* ew, const void* eb,
                             const void* alpha, const void* nw, const void* nb, int T, int W, int V, cudaStream_t s) {
  if (T <= 0) return 0;
  return dtype == 0 ? embed_dyt<float>(ids, w, 1.f, x, h, alpha, nw, nb, ealpha, ew, eb, T, W, V, s)
                    : embed_dyt<bf16>(ids, w, 1.f, x, h, alpha, nw, nb, ealpha, ew, eb, T, W, V, s);
}
extern "C" int vb_dyt(int dtype, const float* x, void* h, const void* alpha, const void* nw, const void* nb, int T, int W, cudaStream_t s) {
  return vb_embed_dyt(dtype, nullptr, nullptr, 1.f, const_cast<float*>(x), h, alpha, nw, nb, T, W, 0, s);
}

extern "C" int vb_rope_pairs(int dtype, void* x, const int* pos, const float* cos_t, const float* sin_t, int T, int heads, long long ld,
                             int hstride, int off, int dims, int max_pos, cudaStream_t s) {
  const int half = dims / 2;
  const long long total = static_cast<long long>(T) * heads * half;
  if (total <= 0) return 0;
  const int grid = static_cast<int>((total + 255) / 256);
  if (dtype == 0) rope_pairs_kernel<float><<<grid, 256, 0, s>>>((float*)x, pos, cos_t, sin_t, heads, ld, hstride, off, half, max_pos, total);
  else rope_pairs_kernel<bf16><<<grid, 256, 0, s>>>((bf16*)x, pos, cos_t, sin_t, heads, ld, hstride, off, half, max_pos, total);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_rope_copy(int dtype, const void* a, long long lda, int a_head, int a_off, void* out, long long ldo, int o_head, int o_off,
                            const int* pos, const float* cos_t, const float* sin_t, int T, int heads, int rot, int half, int max_pos, cudaStream_t s) {
  const long long total = static_cast<long long>(T) * heads * rot;
  if (total <= 0) return 0;
  const int grid = static_cast<int>((total + 255) / 256);
  if (dtype == 0)
    rope_copy_kernel<float><<<grid, 256, 0, s>>>((const float*)a, lda, a_head, a_off, (float*)out, ldo, o_head, o_off, pos, cos_t, sin_t, heads, rot, half, max_pos, total);
  else
    rope_copy_kernel<bf16><<<grid, 256, 0, s>>>((const bf16*)a, lda, a_head, a_off, (bf16*)out, ldo, o_head, o_off, pos, cos_t, sin_t, heads, rot, half, max_pos, total);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_latent_prep(int dtype, const void* p, long long ldp, const void* qn, const void* kn, float eps, const int* pos,
                              const float* cos_t, const float* sin_t, int dims, int max_pos, void* cq, void* lat, long long ldl, void* pages,
                              long long page_stride, int block_size, long long num_slots, const long long* slot, int T, int q_rank,
                              int kv_rank, int rot, cudaStream_t s) {
  if (T <= 0) return 0;
  const bool v8 = dtype == 1 && q_rank % 8 == 0 && kv_rank % 8 == 0 && rot % 8 == 0 && ldp % 8 == 0 && ldl % 8 == 0 && page_stride % 8 == 0 &&
                  !((reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(pages) | reinterpret_cast<uintptr_t>(lat)) & 15);
  if (v8 && q_rank == 0 && kv_rank <= 1024 && rot <= 256 && num_slots < (1ll << 31) && !(reinterpret_cast<uintptr_t>(kn) & 15)) {
    const int grid = (T + 7) / 8;
    auto go = [&](auto kern) {
      kern<<<grid, 256, 0, s>>>((const bf16*)p, ldp, (const bf16*)kn, eps, pos, cos_t, sin_t, dims / 2, max_pos, (bf16*)lat, ldl, (bf16*)pages, page_stride, block_size,
                                num_slots, slot, T, kv_rank, rot);
      return static_cast<int>(cudaGetLastError());
    };
    return kv_rank <= 256 ? go(latent_row_kernel<1>) : kv_rank <= 512 ? go(latent_row_kernel<2>) : go(latent_row_kernel<4>);
  }
#define VB_PREP(T_, V_)                                                                                                                     \
  latent_prep_kernel<T_, V_><<<T, 128, 0, s>>>((const T_*)p, ldp, (const T_*)qn, (const T_*)kn, eps, pos, cos_t, sin_t, dims, max_pos, (T_*)cq, \
                                               (T_*)lat, ldl, (T_*)pages, page_stride, block_size, num_slots, slot, q_rank, kv_rank, rot)
  if (dtype == 0) VB_PREP(float, 1);
  else if (v8) VB_PREP(bf16, 8);
  else VB_PREP(bf16, 1);
#undef VB_PREP
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_gather_pages(int dtype, const void* pages, long long page_stride, int block_size, const int* block_table, int max_blocks,
                               const int* cu_k, const int* k_start, int B, int width, void* out, int total, cudaStream_t s) {
  if (total <= 0) return 0;
  if (dtype == 0)
    gather_pages_kernel<float><<<total, 128, 0, s>>>((const float*)pages, page_stride, block_size, block_table, max_blocks, cu_k, k_start, B, width, (float*)out);
  else
    gather_pages_kernel<bf16><<<total, 128, 0, s>>>((const bf16*)pages, page_stride, block_size, block_table, max_blocks, cu_k, k_start, B, width, (bf16*)out);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int vb_mlstm_decode(int dtype, const void* qkvg, long long ldp, const float* gates, long long ldg, const void* ib, const void* fb,
                               float cap, float* state, long long slot_stride, const uint8_t* active, const void* norm, float eps, void* out,
                               long long ldo, int S, int H, int d, int e, cudaStream_t s) {
  if (S <= 0) return 0;
  if (S > 65535) return -1;
  const bool v4 = e % 4 == 0 && slot_stride % 4 == 0 && !(reinterpret_cast<uintptr_t>(state) & 15);
#define VB_DEC(T_, V_) return mlstm_decode<T_, V_>(qkvg, ldp, gates, ldg, ib, fb, cap, state, slot_stride, active, norm, eps, out, ldo, S, H, d, e, s)
  if (dtype == 0) { if (v4 && ldp % 4 == 0 && (2 * H * d) % 4 == 0) VB_DEC(float, 4); VB_DEC(float, 1); }
  if (v4) VB_DEC(bf16, 4);
  VB_DEC(bf16, 1);
#undef VB_DEC
}

extern "C" int vb_mlstm_scan(int dtype, const void* qkvg, long long ldp, const float* gates, long long ldg, const void* ib, const void* fb,
                             float cap, float* state, long long slot_stride, const int* slots, const int* fresh, const int* cu, int B, float* o,
                             int T, int H, int d, int e, cudaStream_t s) {
  if (T <= 0 || B <= 0) return 0;
  if (B > 65535) return -1;
  return dtype == 0 ? mlstm_scan<float>(qkvg, ldp, gates, ldg, ib, fb, cap, state, slot_stride, slots, fresh, cu, B, o, H, d, e, s)
                    : mlstm_scan<bf16>(qkvg, ldp, gates, ldg, ib, fb, cap, state, slot_stride, slots, fresh, cu, B, o, H, d, e, s);
}

extern "C" int vb_mlstm_out(int dtype, const float* o, const void* g, long long ldg, const void* norm, float eps, void* out, long long ldo,
                            int T, int H, int e, cudaStream_t s) {
  if (T <= 0) return 0;
  const long long total = static_cast<long long>(T) * H;
  const int grid = static_cast<int>((total + 7) / 8);
  if (dtype == 0) mlstm_out_kernel<float><<<grid, 256, 0, s>>>(o, (const float*)g, ldg, (const float*)norm, eps, (float*)out, ldo, total, H, e);
  else mlstm_out_kernel<bf16><<<grid, 256, 0, s>>>(o, (const bf16*)g, ldg, (const bf16*)norm, eps, (bf16*)out, ldo, total, H, e);
  return static_cast<int>(cudaGetLastError());
}
