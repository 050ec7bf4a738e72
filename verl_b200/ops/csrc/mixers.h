// C launchers of the mixer-stack kernels (latent and grouped-query attention, mLSTM and lightning recurrences, short convolutions,
// norms, experts, GEMMs with their epilogues).
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
  VB_EPI_RESID = 4,     // X += acc (+ pb when given), or tanh(palpha acc) pw + pb when pw is given (fp32 residual stream); D = tanh(alpha X) nw + nb in the
                        // operands' type when D is given
  VB_EPI_SOFTCAP = 5,   // D = cap * tanh(acc / cap) in the operands' type
  VB_EPI_BIAS = 6,      // D = acc + nb in the operands' type
  VB_EPI_SILU = 7,      // D = silu(acc) in columns [0, n0), acc in the others, in the operands' type
  VB_EPI_BIAS_RELU2 = 8,// D = max(acc + nb, 0)^2 in the operands' type
  VB_EPI_TANH = 9,      // D = acc in columns [0, n0), tanh(acc) in the others, in the operands' type
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
  float cap;
  const float* gate;  // batched products: batch z of row m is multiplied by sigmoid(gate[m * ldg + z]) when given
  long long ldg;
  const void* palpha; // VB_EPI_RESID: norm of the product (scalar, [N], [N]), or null; pb alone: a bias
  const void* pw;
  const void* pb;
};

// Attention with per-head or shared keys and values. Latent attention: du unrotated and dr rotated key dimensions (the latter
// shared by the heads); grouped-query attention: dr = 0, query head h reads key / value head h / kv_group.
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
  int kv_group;             // query heads per key / value head (0 or 1: one)
  float softcap;            // score = softcap * tanh(score / softcap); 0: off
  int keep_first;           // with a window: the sequence's first keys that every query sees besides
  int chunk;                // > 0: a query sees the keys from its chunk's start on; the sequence's first key row starts a chunk
  // maps = 2: differential attention. H counts maps (query map m of head h is 2h + m, key map m of head g is 2g + m) and kv_group the
  // query heads per value head, maps not counted; out [T, H / 2, dv]: (1 - diff) rms_norm(a1 - lambda a2), lambda from the
  // four vectors of du entries at diff_vec (exp(x0 . x1) - exp(x2 . x3) + diff)
  int maps;
  int split_maps;           // vb_latent_prefill: every query head is a map (key head as with maps = 2, maps apart in out [T, H, dv])
  const void* diff_vec;
  float diff, eps;
};

// x += mult * rms_norm(Y) * nw;  Y = [sigmoid(gate)] sum of `splits` planes of y + sum_j rows[slot[t, j]]
struct VbResidRms {
  float* x;                 // [T, W] fp32 residual stream
  const void* y;            // null: none
  int y_f32, splits;        // y in fp32 (partial products) or in the weights' type (one plane)
  long long split_stride, ldy;
  const void* rows;         // expert outputs, or null
  long long ldr;
  const int* slot;          // [T, top]
  int top;
  const float* gate;        // gate[t * ldgate], or null
  long long ldgate;
  const void *nw, *next;    // norm of the sublayer; next: norm of the new stream, or null (h is the stream itself)
  void* h;                  // [T, W]
  float eps, mult;
  int T, W;
};

struct VbQkvPrep {
  const void* p; long long ldp;       // [T, q | k | v]
  const void *qn, *kn;                // [dim]
  const int* pos;
  const float *cos_t, *sin_t;         // [max_pos, half]
  int half, max_pos;
  const void* vfirst; long long ldvf; // values of the first mixing layer (or null)
  const void* vmix;                   // scalar
  void* q;                            // [T, H, dim]
  void* rows; long long ldr;          // [T, G (dim + vdim)] or null
  void* pages; long long page_stride; int block_size; long long num_slots; const long long* slot;
  int T, H, G, dim, vdim;
  float eps;
};

// x += post(sum_j rows[slot[t, j]]), h = next(x); both norms Dynamic Tanh
struct VbResidDyt {
  float* x;                 // [T, W]
  const void* rows; long long ldr;
  const int* slot; int top; // [T, top]
  const void *palpha, *pw, *pb, *alpha, *nw, *nb;
  void* h;                  // [T, W]
  int T, W;
};

// Row p[t] = [q of H heads | k of G heads | v of GV heads]: causal convolution per channel, rotation of q and k, norm without weight.
struct VbConvPrep {
  const void* p; long long ldp;
  const void* conv; int taps;         // [channels, taps], last tap = the token itself (null: no convolution, taps = 1)
  const int* cu; int B;               // portions: sequence b = tokens cu[b] .. cu[b + 1]; null: one token per sequence
  float* state; long long slot_stride;// last taps - 1 inputs per slot, [taps - 1, channels], oldest first (null: zeros, nothing kept)
  const int *slots, *fresh;           // portions
  const uint8_t* active;              // steps: row t is slot t
  const int* pos; const float *cos_t, *sin_t; int half, max_pos, halves;
  void* q;                            // [T, H, dim]
  void* rows; long long ldr;          // [T, G dim + GV vdim] or null
  void* pages; long long page_stride; int block_size; long long num_slots; const long long* page_slot;
  int T, H, G, GV, dim, vdim, norm;   // norm 0: none
  float eps;
};

// Row p[t] = [q | k | v]: weighted RMS norms over all query and over all key columns, queries times temp of their head.
struct VbWholeNorm {
  const void* p; long long ldp;
  const void *qn, *kn, *temp;         // [H dim], [G dim], [H]
  void* q;                            // [T, H dim]
  void* rows; long long ldr;          // [T, G (dim + vdim)] or null
  void* pages; long long page_stride; int block_size; long long num_slots; const long long* page_slot;
  int T, H, G, dim, vdim;
  float eps;
};

// h = rms_norm(x) nw, plus its causal convolution over time with `conv` [W, taps] when given (last tap: the token itself).
struct VbRmsConv {
  float* x;                           // [T, W]; first x += sum of `splits` planes of y (+ bias) when given (steps only)
  const void* y; int y_f32, splits; long long split_stride, ldy;
  const void *bias, *nw, *conv;
  int taps;
  const int* cu; int B;               // portions; null: one token per slot
  float* state; long long slot_stride;// last taps - 1 rows of a sequence, [taps - 1, W], oldest first
  const int *slots, *fresh;
  const uint8_t* active;
  void* h;                            // [T, W]
  int T, W;
  float eps;
};

// Generalized delta rule over rows p[t] = [r | k | v | za | g | ...] (H d columns each): S = diag(w) S - (a u)(u^T S) + k v^T, o = S^T r with
// w = exp(-exp(-1/2) sigmoid(zw + w0)), a = sigmoid(za + ab), u = k / sqrt(k . k + 1e-6).
struct VbDelta {
  const void* p; long long ldp;
  const void* zw; long long ldz;      // [T, H d]
  const void *ab, *w0;                // [H d]
  float* state; long long slot_stride;// [slots, H, d, d] or null
  const int *slots, *fresh, *cu;      // portions
  const uint8_t* active;              // steps: row t is slot t
  const void* norm; float eps;        // steps: out = rms_norm(o) norm sigmoid(g)
  void* out; long long ldo;           // [T, H d]
  int T, B, H, d;
};

// Recurrence S = decay S + k v^T, o = S^T q per head over rows p[t] = [q | k | v | ...].
struct VbLightning {
  const void* p; long long ldp;
  const float* decay;                 // [H]
  float* state; long long slot_stride;// [slots, H, d, e] or null
  const int *slots, *fresh, *cu;      // portions
  const uint8_t* active;              // steps: row t is slot t
  void* out; long long ldo;           // [T, H e]
  int T, B, H, d, e;
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
// rows grouped by expert: 128-row tile i of A meets B[tile_expert[i]] ([N, K] matrices, back to back); tiles past *num_tiles are skipped
int vb_gemm_simt_grouped(int dtype, const void* A, const void* B, int M, int N, int K, long long lda, const int* tile_expert, const int* num_tiles,
                         const VbEpiArgs* e, cudaStream_t s);
// gemm_tcgen05.cu / gemm_skinny_tcgen05.cu: same epilogues on the tensor cores (bf16). Return -1 for shapes they do not serve.
int vb_gemm_bf16_epi(const void* A, const void* B, int M, int N, int K, long long lda, long long ldb, const VbEpiArgs* e, cudaStream_t s);
int vb_gemm_skinny_epi(const void* X, const void* W, int M, int N, int K, long long ldx, long long ldw, const VbEpiArgs* e, int splits,
                       float* ws, cudaStream_t s);
// act[rows, I] = silu(r g) * (r u), [g | u] = A W_e^T with W_e = [gate; up] ([2I, K]) of the tile's expert and r = row_scale[row];
// clip > 0: r g sigmoid(1.702 g) (u + 1) with g <= clip and |u| <= clip
int vb_gemm_grouped_swiglu(const void* A, const void* W, void* act, int rows_cap, int I, int K, long long lda, long long ldd, const float* row_scale,
                           int E, const int* tile_expert, const int* num_tiles, float clip, cudaStream_t s);
// stack_rows.cu
int vb_embed_rms(int dtype, const long long* ids, const void* w, float scale, const void* nw, float eps, float* x, void* h, int T, int W, int V,
                 cudaStream_t s);
int vb_residual_rms(int dtype, const VbResidRms* p, cudaStream_t s);
int vb_gated_silu(int dtype, const void* gu, long long ldg, const float* row_scale, float clip, void* out, int T, int I, cudaStream_t s);
int vb_residual_dyt(int dtype, const VbResidDyt* p, cudaStream_t s);
// W = heads * size: statistics over each head's columns
int vb_gated_rms(int dtype, const void* o, long long ldo, const void* g, long long ldg, const void* norm, float eps, void* out, int T, int W, int heads,
                 cudaStream_t s);
// x[t, c] = tanh(x[t, c]) for c < n
int vb_tanh_cols(int dtype, void* x, long long ld, int T, int n, cudaStream_t s);
int vb_whole_norm(int dtype, const VbWholeNorm* p, cudaStream_t s);
// a [T, 2 H, dv] -> out [T, H, dv], see VbLatentAttn::maps
int vb_diff_combine(int dtype, const void* a, int a_f32, const void* vec, int dim, float diff, float eps, void* out, int T, int H, int dv, cudaStream_t s);
// rms_conv.cu
int vb_embed_rows(int dtype, const long long* ids, const void* w, float scale, float* x, int T, int W, int V, cudaStream_t s);
int vb_rms_conv(int dtype, const VbRmsConv* p, cudaStream_t s);
// delta_rule.cu / delta_chunk.cu
int vb_delta_decode(int dtype, const VbDelta* p, cudaStream_t s);
int vb_delta_scan(int dtype, const VbDelta* p, cudaStream_t s);
int vb_delta_chunk_segments(const VbDelta* p);
int vb_delta_chunk(const VbDelta* p, int nseg, float* ws, cudaStream_t s);
// conv_prep.cu
int vb_conv_prep(int dtype, const VbConvPrep* p, cudaStream_t s);
// lightning.cu / lightning_tcgen05.cu (d <= 128) / lightning_chunk.cu; nseg > 1: workspace of B (nseg - 1) H d e floats
int vb_lightning_decode(int dtype, const VbLightning* p, cudaStream_t s);
int vb_lightning_scan(int dtype, const VbLightning* p, cudaStream_t s);
int vb_lightning_chunk_segments(int T, int B, int H, int d, int e, int all_fresh);
int vb_lightning_tc(const VbLightning* p, int nseg, float* local, cudaStream_t s);
int vb_lightning_chunk(const VbLightning* p, int nseg, float* local, cudaStream_t s);
int vb_qkv_prep(int dtype, const VbQkvPrep* p, cudaStream_t s);
// experts.cu
// corr (null: none) is added to the scores for the choice; groups > 1: only experts of the `keep` best groups can be chosen
int vb_expert_route(int dtype, const float* z, long long ldz, const void* corr, int groups, int keep, int T, int E, int k, int renorm, float* score, int* expert, int* rank, int* counts, cudaStream_t s);
int vb_expert_place(int dtype, const void* h, long long ldh, const float* score, const int* expert, const int* rank, const int* counts, int T, int E, int k,
                    int W, void* x, float* row_scale, int* slot, int* tile_expert, int* num_tiles, int max_tiles, cudaStream_t s);
// grouped_decode.cu
int vb_grouped_decode_splits(const VbLatentAttn* a, int max_keys);
int vb_grouped_decode(const VbLatentAttn* a, long long num_blocks, int nsplit, float* part_o, float* part_ml, cudaStream_t s);
// mixer_kernels.cu
int vb_embed_dyt(int dtype, const long long* ids, const void* w, float scale, float* x, void* h, const void* alpha, const void* nw,
                 const void* nb, int T, int W, int V, cudaStream_t s);
// x = tanh(ealpha w[id]) ew + eb, h = tanh(alpha x) nw + nb
int vb_embed_dyt2(int dtype, const long long* ids, const void* w, float* x, void* h, const void* ealpha, const void* ew, const void* eb, const void* alpha,
                  const void* nw, const void* nb, int T, int W, int V, cudaStream_t s);
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
// out_f32: out is fp32 whatever the operands' type
int vb_latent_attn_simt(int dtype, const VbLatentAttn* a, int out_f32, cudaStream_t s);
}
