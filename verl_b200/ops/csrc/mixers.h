// C launchers of the mixer-stack kernels (latent attention, mLSTM, Dynamic Tanh, GEMMs with their epilogues).
// dtype: 0 = fp32 tensors, 1 = bf16 tensors (weights and activations; statistics, states and residual are always fp32).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

// What a GEMM does with its accumulator (acc = A B^T).
enum VbEpi : int {
  VB_EPI_STORE = 0,     // D = acc in the operands' type
  VB_EPI_STORE_F32 = 1, // D = acc as fp32
  VB_EPI_GELU = 2,      // D = erf-gelu(acc) in the operands' type
  VB_EPI_SPLIT = 3,     // columns [0, n0) -> D in the operands' type, columns [n0, N) -> D2 as fp32
  VB_EPI_RESID = 4,     // X += acc (fp32 residual stream); D = tanh(alpha X) w + b in the operands' type when D is given
};

struct VbEpiArgs {
  int mode;
  void* D;
  long long ldd;
  int n0;
  float* D2;
  long long ldd2;
  float* X;
  long long ldx;
  const void* alpha;  // scalar, operands' type
  const void* nw;     // [N]
  const void* nb;     // [N]
  const float* gate;  // batched products: batch z of row m is multiplied by sigmoid(gate[m * ldg + z]) when given
  long long ldg;
};

struct VbLatentAttn {
  // queries [T, H, du + dr]: row stride ldq, head stride hq; unrotated part first
  const void* q; long long ldq; int hq;
  // keys / values: element (row, head, i) at ku[row * ku_row + head * ku_head + i] (and kr without heads)
  const void* ku; long long ku_row; int ku_head;
  const void* kr; long long kr_row;
  const void* v; long long v_row; int v_head;
  // rows: contiguous per sequence (cu_k) or through a page table
  const int* cu_q;          // [B + 1] query rows per sequence (null: one query per sequence)
  const int* cu_k;          // [B + 1] key rows per sequence, the last key belongs to the last query (null: paged)
  const int* block_table; int max_blocks; int block_size; long long page_stride;  // rows per page step (in rows)
  const int* ctx_len;       // [B] paged: keys of the sequence (0: inactive, output zero)
  const float* gate; long long ldg;  // output multiplied by sigmoid(gate[t, h]) when given
  const void* sink;         // [H] or null
  void* out; long long ldo; // [T, H, dv]
  int B, T, H, du, dr, dv, window;
  float scale;
};

struct VbHeadwise {
  const void* a; long long lda, a_head;   // a[m, h, k]
  const void* w; long long w_head, ldw;   // w[h] as [N, K] (kn = 0) or [K, N] (kn = 1)
  int kn;
  void* out; long long ldo, o_head;
  int M, N, K, H;
  const float* gate; long long ldg;
  // rot > 0: a[m, h, K .. K + rot) is rotated (pairs of the first 2 * half dimensions) and stored behind the product
  int rot, half, max_pos;
  const int* pos;
  const float *cos_t, *sin_t;
};

extern "C" {
void verl_count_launches(long long n);
// gemm_simt.cu
int vb_gemm_simt(int dtype, const void* A, const void* B, int M, int N, int K, long long lda, long long ldb, int b_mn, int batch,
                 long long sa, long long sb, long long sd, const VbEpiArgs* e, cudaStream_t s);
// gemm_tcgen05.cu / gemm_skinny_tcgen05.cu: same epilogues on the tensor cores (bf16). Return -1 for shapes they do not serve.
int vb_gemm_bf16_epi(const void* A, const void* B, int M, int N, int K, long long lda, long long ldb, const VbEpiArgs* e, cudaStream_t s);
int vb_gemm_skinny_epi(const void* X, const void* W, int M, int N, int K, long long ldx, long long ldw, const VbEpiArgs* e, int splits,
                       float* ws, cudaStream_t s);
// mixer_kernels.cu
int vb_embed_dyt(int dtype, const long long* ids, const void* w, float scale, float* x, void* h, const void* alpha, const void* nw,
                 const void* nb, int T, int W, int V, cudaStream_t s);
int vb_dyt(int dtype, const float* x, void* h, const void* alpha, const void* nw, const void* nb, int T, int W, cudaStream_t s);
int vb_rope_pairs(int dtype, void* x, const int* pos, const float* cos_t, const float* sin_t, int T, int heads, long long ld, int hstride,
                  int off, int dims, int max_pos, cudaStream_t s);
int vb_rope_copy(int dtype, const void* a, long long lda, int a_head, int a_off, void* out, long long ldo, int o_head, int o_off, const int* pos,
                 const float* cos_t, const float* sin_t, int T, int heads, int rot, int half, int max_pos, cudaStream_t s);
int vb_latent_prep(int dtype, const void* p, long long ldp, const void* qn, const void* kn, float eps, const int* pos, const float* cos_t,
                   const float* sin_t, int dims, int max_pos, void* cq, void* lat, long long ldl, void* pages, long long page_stride,
                   int block_size, long long num_slots, const long long* slot, int T, int q_rank, int kv_rank, int rot, cudaStream_t s);
int vb_gather_pages(int dtype, const void* pages, long long page_stride, int block_size, const int* block_table, int max_blocks,
                    const int* cu_k, const int* k_start, int B, int width, void* out, int total, cudaStream_t s);
int vb_mlstm_decode(int dtype, const void* qkvg, long long ldp, const float* gates, long long ldg, const void* ib, const void* fb, float cap,
                    float* state, long long slot_stride, const uint8_t* active, const void* norm, float eps, void* out, long long ldo, int S,
                    int H, int d, int e, cudaStream_t s);
int vb_mlstm_scan(int dtype, const void* qkvg, long long ldp, const float* gates, long long ldg, const void* ib, const void* fb, float cap,
                  float* state, long long slot_stride, const int* slots, const int* fresh, const int* cu, int B, float* o, int T, int H, int d,
                  int e, cudaStream_t s);
int vb_mlstm_out(int dtype, const float* o, const void* g, long long ldg, const void* norm, float eps, void* out, long long ldo, int T, int H,
                 int e, cudaStream_t s);
// latent_prefill_tcgen05.cu
int vb_latent_prefill(const VbLatentAttn* a, int Tk, cudaStream_t s);
// mlstm_chunk.cu
int vb_mlstm_chunk_segments(int T, int B, int H, int d, int e, int all_fresh);
int vb_mlstm_chunk(const void* qkvg, long long ldp, const float* gates, long long ldg, const void* ib, const void* fb, float cap, float* state,
                   long long slot_stride, const int* slots, const int* fresh, const int* cu, int B, int nseg, float* local, const void* norm,
                   float eps, void* out, long long ldo, int H, int d, int e, cudaStream_t s);
// headwise_mma.cu
int vb_headwise(const VbHeadwise* p, cudaStream_t s);
// latent_decode.cu
int vb_latent_decode_splits(int S, int H, int rank, int width, int block_size, int max_keys);
int vb_latent_decode(const VbLatentAttn* a, long long num_blocks, int nsplit, float* part_o, float* part_ml, cudaStream_t s);
// latent_attention_simt.cu
int vb_latent_attn_simt(int dtype, const VbLatentAttn* a, cudaStream_t s);
}
