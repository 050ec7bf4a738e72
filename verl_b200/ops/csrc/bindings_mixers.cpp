// torch.ops.verl_b200.* bindings of the mixer-stack kernels.
#include <ATen/ATen.h>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/library.h>

#include "launchers.h"
#include "mixers.h"

namespace {

using at::Tensor;
using OptTensor = c10::optional<at::Tensor>;

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }
inline void* ptr(const OptTensor& t) { return t.has_value() ? t->data_ptr() : nullptr; }
inline int* iptr(const OptTensor& t) { return t.has_value() ? t->data_ptr<int>() : nullptr; }
inline const long long* lptr(const Tensor& t) { return reinterpret_cast<const long long*>(t.data_ptr<int64_t>()); }
int dtype_of(const Tensor& t) {
  TORCH_CHECK(t.is_cuda(), "expected a CUDA tensor");
  if (t.scalar_type() == at::kFloat) return 0;
  TORCH_CHECK(t.scalar_type() == at::kBFloat16, "expected an fp32 or bf16 tensor");
  return 1;
}
void same(const Tensor& a, const Tensor& b, const char* what) { TORCH_CHECK(b.is_cuda() && a.scalar_type() == b.scalar_type(), what, ": types differ"); }
#define CHECK_RC(rc, what) TORCH_CHECK((rc) == 0, what " failed with code ", (rc))
#define CHECK_F32(x) TORCH_CHECK((x).is_cuda() && (x).scalar_type() == at::kFloat, #x " must be a CUDA fp32 tensor")
#define CHECK_I32(x) TORCH_CHECK((x).is_cuda() && (x).scalar_type() == at::kInt && (x).is_contiguous(), #x " must be a contiguous int32 CUDA tensor")

// D = epilogue(a w^T): tensor cores where the sizes allow, the fp32-pipeline kernel otherwise.
void run_gemm(const Tensor& a, const Tensor& w, const VbEpiArgs& e) {
  const int dt = dtype_of(a);
  same(a, w, "linear");
  TORCH_CHECK(a.dim() == 2 && w.dim() == 2 && a.stride(1) == 1 && w.stride(1) == 1 && a.size(1) == w.size(1), "linear: a [M, K], w [N, K]");
  const int M = (int)a.size(0), K = (int)a.size(1), N = (int)w.size(0);
  if (M == 0 || N == 0) return;
  verl_count_launches(1);
  int rc = -1;
  if (dt == 1) {
    if (M <= 1024 && N % 8 == 0 && K % 8 == 0 && a.stride(0) % 8 == 0 && w.stride(0) % 8 == 0) {
      const int s = vb_gemm_skinny_splits(M, N, K);
      if (s >= 1) {
        Tensor ws;
        if (s > 1) ws = at::empty({s, M, N}, a.options().dtype(at::kFloat));
        rc = vb_gemm_skinny_epi(a.data_ptr(), w.data_ptr(), M, N, K, a.stride(0), w.stride(0), &e, s, s > 1 ? ws.data_ptr<float>() : nullptr, cur_stream());
      }
    }
    if (rc < 0 && e.mode == VB_EPI_STORE && e.gate == nullptr && M > 1024 && N % 8 == 0 && K % 8 == 0 && a.stride(0) % 8 == 0 && w.stride(0) % 8 == 0 && e.ldd % 8 == 0 &&
        !((reinterpret_cast<uintptr_t>(a.data_ptr()) | reinterpret_cast<uintptr_t>(w.data_ptr()) | reinterpret_cast<uintptr_t>(e.D)) & 15))
      rc = vb_gemm_bf16(a.data_ptr(), w.data_ptr(), e.D, nullptr, M, N, K, a.stride(0), w.stride(0), e.ldd, 0, 0, 0, 0, 0, cur_stream());
    if (rc < 0) rc = vb_gemm_bf16_epi(a.data_ptr(), w.data_ptr(), M, N, K, a.stride(0), w.stride(0), &e, cur_stream());
  }
  if (rc < 0) rc = vb_gemm_simt(dt, a.data_ptr(), w.data_ptr(), M, N, K, a.stride(0), w.stride(0), 0, 1, 0, 0, 0, &e, cur_stream());
  TORCH_CHECK(rc == 0, "linear with epilogue ", e.mode, " failed with code ", rc, " (M=", M, " N=", N, " K=", K, ")");
}

Tensor linear_act(const Tensor& a, const Tensor& w, bool gelu, bool out_f32) {
  const c10::cuda::CUDAGuard guard(a.device());
  Tensor d = at::empty({a.size(0), w.size(0)}, out_f32 ? a.options().dtype(at::kFloat) : a.options());
  VbEpiArgs e{};
  e.mode = gelu ? VB_EPI_GELU : (out_f32 ? VB_EPI_STORE_F32 : VB_EPI_STORE);
  e.D = d.data_ptr(); e.ldd = d.stride(0);
  run_gemm(a, w, e);
  return d;
}

std::tuple<Tensor, Tensor> linear_split(const Tensor& a, const Tensor& w, int64_t n0) {
  const c10::cuda::CUDAGuard guard(a.device());
  const int64_t M = a.size(0), N = w.size(0);
  TORCH_CHECK(n0 > 0 && n0 < N, "linear_split: 0 < n0 < N");
  Tensor d = at::empty({M, n0}, a.options()), d2 = at::empty({M, N - n0}, a.options().dtype(at::kFloat));
  VbEpiArgs e{};
  e.mode = VB_EPI_SPLIT;
  e.D = d.data_ptr(); e.ldd = n0; e.n0 = (int)n0; e.D2 = d2.data_ptr<float>(); e.ldd2 = N - n0;
  run_gemm(a, w, e);
  return {d, d2};
}

Tensor linear_bias(const Tensor& a, const Tensor& w, const Tensor& b, bool relu2) {
  const c10::cuda::CUDAGuard guard(a.device());
  same(a, b, "linear_bias");
  TORCH_CHECK(b.numel() == w.size(0) && b.is_contiguous(), "linear_bias: bias [N]");
  Tensor d = at::empty({a.size(0), w.size(0)}, a.options());
  VbEpiArgs e{};
  e.mode = relu2 ? VB_EPI_BIAS_RELU2 : VB_EPI_BIAS;
  e.D = d.data_ptr(); e.ldd = d.stride(0); e.nb = b.data_ptr();
  run_gemm(a, w, e);
  return d;
}

Tensor linear_tanh(const Tensor& a, const Tensor& w, int64_t n0) {
  const c10::cuda::CUDAGuard guard(a.device());
  Tensor d = at::empty({a.size(0), w.size(0)}, a.options());
  TORCH_CHECK(n0 >= 0 && n0 <= w.size(0), "linear_tanh: 0 <= n0 <= N");
  VbEpiArgs e{};
  // few tokens: the plain product of the decode kernel and a small launch for the few columns beat its epilogue with a function
  const bool apart = dtype_of(a) == 1 && a.size(0) <= 1024 && n0 >= w.size(0) / 2;
  e.mode = apart ? VB_EPI_STORE : VB_EPI_TANH;
  e.D = d.data_ptr(); e.ldd = d.stride(0); e.n0 = (int)n0;
  run_gemm(a, w, e);
  if (apart && n0 < w.size(0)) {
    verl_count_launches(1);
    CHECK_RC(vb_tanh_cols(1, reinterpret_cast<char*>(d.data_ptr()) + n0 * d.element_size(), d.stride(0), (int)d.size(0), (int)(w.size(0) - n0), cur_stream()), "vb_tanh_cols");
  }
  return d;
}

Tensor linear_silu(const Tensor& a, const Tensor& w, int64_t n0) {
  const c10::cuda::CUDAGuard guard(a.device());
  Tensor d = at::empty({a.size(0), w.size(0)}, a.options());
  VbEpiArgs e{};
  e.mode = VB_EPI_SILU;
  e.D = d.data_ptr(); e.ldd = d.stride(0); e.n0 = (int)n0;
  run_gemm(a, w, e);
  return d;
}

// x += a w^T (+ bias), or x += tanh(palpha a w^T) pw + pb (fp32 residual stream); returns tanh(alpha x) nw + nb in a's type, or an empty tensor
// without a norm.
Tensor linear_residual_(const Tensor& a, const Tensor& w, Tensor x, const OptTensor& alpha, const OptTensor& nw, const OptTensor& nb, const OptTensor& palpha,
                        const OptTensor& pw, const OptTensor& pb, const OptTensor& bias) {
  const c10::cuda::CUDAGuard guard(a.device());
  CHECK_F32(x);
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && x.size(0) == a.size(0) && x.size(1) == w.size(0), "linear_residual_: x [M, N]");
  VbEpiArgs e{};
  e.mode = VB_EPI_RESID;
  e.X = x.data_ptr<float>(); e.ldx = x.stride(0);
  Tensor h;
  if (nw.has_value()) {
    same(a, *nw, "linear_residual_");
    same(a, *nb, "linear_residual_");
    same(a, *alpha, "linear_residual_");
    TORCH_CHECK(nw->numel() == w.size(0) && nb->numel() == w.size(0) && alpha->numel() == 1, "linear_residual_: norm sizes");
    h = at::empty({a.size(0), w.size(0)}, a.options());
    e.D = h.data_ptr(); e.ldd = h.stride(0); e.alpha = alpha->data_ptr(); e.nw = nw->data_ptr(); e.nb = nb->data_ptr();
  } else {
    h = at::empty({0}, a.options());
  }
  if (pw.has_value()) {
    same(a, *pw, "linear_residual_");
    same(a, *pb, "linear_residual_");
    same(a, *palpha, "linear_residual_");
    TORCH_CHECK(pw->numel() == w.size(0) && pb->numel() == w.size(0) && palpha->numel() == 1, "linear_residual_: norm sizes");
    e.palpha = palpha->data_ptr(); e.pw = pw->data_ptr(); e.pb = pb->data_ptr();
  }
  if (bias.has_value()) {
    same(a, *bias, "linear_residual_");
    TORCH_CHECK(!pw.has_value() && bias->numel() == w.size(0) && bias->is_contiguous(), "linear_residual_: bias [N]");
    e.pb = bias->data_ptr();
  }
  run_gemm(a, w, e);
  return h;
}

std::tuple<Tensor, Tensor> embed_dyt(const Tensor& ids, const Tensor& w, double scale, const Tensor& alpha, const Tensor& nw, const Tensor& nb) {
  const int dt = dtype_of(w);
  const c10::cuda::CUDAGuard guard(w.device());
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous() && w.is_contiguous() && nw.numel() == w.size(1), "embed_dyt");
  same(w, nw, "embed_dyt");
  const int T = (int)ids.numel(), W = (int)w.size(1);
  Tensor x = at::empty({T, W}, w.options().dtype(at::kFloat)), h = at::empty({T, W}, w.options());
  verl_count_launches(1);
  CHECK_RC(vb_embed_dyt(dt, lptr(ids), w.data_ptr(), (float)scale, x.data_ptr<float>(), h.data_ptr(), alpha.data_ptr(), nw.data_ptr(),
                        nb.data_ptr(), T, W, (int)w.size(0), cur_stream()), "vb_embed_dyt");
  return {x, h};
}

std::tuple<Tensor, Tensor> embed_dyt2(const Tensor& ids, const Tensor& w, const Tensor& ealpha, const Tensor& ew, const Tensor& eb, const Tensor& alpha,
                                      const Tensor& nw, const Tensor& nb) {
  const int dt = dtype_of(w);
  const c10::cuda::CUDAGuard guard(w.device());
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous() && w.is_contiguous() && nw.numel() == w.size(1) && nb.numel() == w.size(1) &&
              ew.numel() == w.size(1) && eb.numel() == w.size(1) && ealpha.numel() == 1 && alpha.numel() == 1, "embed_dyt2");
  for (const Tensor* t : {&nw, &nb, &alpha, &ew, &eb, &ealpha}) same(w, *t, "embed_dyt2");
  const int T = (int)ids.numel(), W = (int)w.size(1);
  Tensor x = at::empty({T, W}, w.options().dtype(at::kFloat)), h = at::empty({T, W}, w.options());
  verl_count_launches(1);
  CHECK_RC(vb_embed_dyt2(dt, lptr(ids), w.data_ptr(), x.data_ptr<float>(), h.data_ptr(), ealpha.data_ptr(), ew.data_ptr(), eb.data_ptr(), alpha.data_ptr(),
                         nw.data_ptr(), nb.data_ptr(), T, W, (int)w.size(0), cur_stream()), "vb_embed_dyt2");
  return {x, h};
}

// x += post(sum_j rows[slot[t, j]]); returns norm(x) in the norm's type (both Dynamic Tanh).
Tensor residual_dyt_(Tensor x, const Tensor& rows, const Tensor& slot, const Tensor& palpha, const Tensor& pw, const Tensor& pb, const Tensor& alpha, const Tensor& nw,
                     const Tensor& nb) {
  CHECK_F32(x);
  CHECK_I32(slot);
  const int dt = dtype_of(nw);
  const c10::cuda::CUDAGuard guard(x.device());
  for (const Tensor* t : {&rows, &palpha, &pw, &pb, &alpha, &nb}) same(nw, *t, "residual_dyt_");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && rows.dim() == 2 && rows.stride(1) == 1 && rows.size(1) == x.size(1) && slot.dim() == 2 && slot.size(0) == x.size(0) &&
              nw.numel() == x.size(1) && nb.numel() == x.size(1) && pw.numel() == x.size(1) && pb.numel() == x.size(1) && alpha.numel() == 1 && palpha.numel() == 1,
              "residual_dyt_: sizes");
  VbResidDyt p{};
  p.x = x.data_ptr<float>(); p.rows = rows.data_ptr(); p.ldr = rows.stride(0); p.slot = slot.data_ptr<int>(); p.top = (int)slot.size(1);
  p.palpha = palpha.data_ptr(); p.pw = pw.data_ptr(); p.pb = pb.data_ptr(); p.alpha = alpha.data_ptr(); p.nw = nw.data_ptr(); p.nb = nb.data_ptr();
  p.T = (int)x.size(0); p.W = (int)x.size(1);
  Tensor h = at::empty({p.T, p.W}, nw.options());
  p.h = h.data_ptr();
  verl_count_launches(1);
  CHECK_RC(vb_residual_dyt(dt, &p, cur_stream()), "vb_residual_dyt");
  return h;
}

// rms_norm(o) norm sigmoid(g) over whole rows or each of `heads` parts (strided views).
Tensor gated_rms(const Tensor& o, const Tensor& g, const Tensor& norm, double eps, int64_t heads) {
  const int dt = dtype_of(o);
  same(o, g, "gated_rms");
  same(o, norm, "gated_rms");
  TORCH_CHECK(o.dim() == 2 && g.sizes() == o.sizes() && o.stride(1) == 1 && g.stride(1) == 1 && norm.numel() == o.size(1) && heads >= 1 &&
              o.size(1) % heads == 0, "gated_rms: [T, W]");
  const c10::cuda::CUDAGuard guard(o.device());
  Tensor out = at::empty(o.sizes(), o.options());
  verl_count_launches(1);
  CHECK_RC(vb_gated_rms(dt, o.data_ptr(), o.stride(0), g.data_ptr(), g.stride(0), norm.data_ptr(), (float)eps, out.data_ptr(), (int)o.size(0), (int)o.size(1),
                        (int)heads, cur_stream()), "vb_gated_rms");
  return out;
}

Tensor dynamic_tanh(const Tensor& x, const Tensor& alpha, const Tensor& nw, const Tensor& nb) {
  CHECK_F32(x);
  const int dt = dtype_of(nw);
  const c10::cuda::CUDAGuard guard(x.device());
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && nw.numel() == x.size(1) && nb.numel() == x.size(1) && alpha.numel() == 1, "dynamic_tanh");
  Tensor h = at::empty(x.sizes(), nw.options());
  verl_count_launches(1);
  CHECK_RC(vb_dyt(dt, x.data_ptr<float>(), h.data_ptr(), alpha.data_ptr(), nw.data_ptr(), nb.data_ptr(), (int)x.size(0), (int)x.size(1), cur_stream()), "vb_dyt");
  return h;
}

// In-place rotation of pairs (off + 2i, off + 2i + 1) of every head of x [T, heads, n] (a strided view), i < dims / 2.
void rope_pairs_(Tensor x, const Tensor& pos, const Tensor& cs, const Tensor& sn, int64_t off, int64_t dims) {
  const int dt = dtype_of(x);
  CHECK_I32(pos);
  CHECK_F32(cs);
  CHECK_F32(sn);
  TORCH_CHECK(x.dim() == 3 && x.stride(2) == 1 && off >= 0 && off + dims <= x.size(2) && dims % 2 == 0 && cs.size(1) == dims / 2 && cs.is_contiguous() &&
              sn.is_contiguous() && pos.numel() == x.size(0), "rope_pairs_");
  const c10::cuda::CUDAGuard guard(x.device());
  verl_count_launches(1);
  CHECK_RC(vb_rope_pairs(dt, x.data_ptr(), pos.data_ptr<int>(), cs.data_ptr<float>(), sn.data_ptr<float>(), (int)x.size(0), (int)x.size(1), x.stride(0),
                         (int)x.stride(1), (int)off, (int)dims, (int)cs.size(0), cur_stream()), "vb_rope_pairs");
}

// p [T, q_rank + kv_rank + rot]; pages: view [blocks, block_size, kv_rank + rot] of the cache (or none), slot int64 [T] (negative: no append).
std::tuple<Tensor, Tensor> latent_prep(const Tensor& p, const OptTensor& qn, const Tensor& kn, double eps, const Tensor& pos, const Tensor& cs,
                                       const Tensor& sn, const OptTensor& pages, const OptTensor& slot, bool want_rows) {
  const int dt = dtype_of(p);
  CHECK_I32(pos);
  if (qn.has_value()) same(p, *qn, "latent_prep");
  same(p, kn, "latent_prep");
  const int64_t T = p.size(0), qr = qn.has_value() ? qn->numel() : 0, kr = kn.numel(), rot = p.size(1) - qr - kr;
  TORCH_CHECK(p.stride(1) == 1 && rot >= 0 && pos.numel() == T && cs.is_contiguous() && sn.is_contiguous() && 2 * cs.size(1) <= std::max<int64_t>(rot, 0), "latent_prep: sizes");
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor cq = at::empty({T, qr}, p.options());
  Tensor lat = at::empty({want_rows ? T : 0, kr + rot}, p.options());
  long long ps = 0, slots = 0;
  int bs = 1;
  if (pages.has_value()) {
    same(p, *pages, "latent_prep");
    TORCH_CHECK(pages->dim() == 3 && pages->size(2) == kr + rot && pages->stride(2) == 1 && pages->stride(1) == kr + rot && slot.has_value() &&
                slot->scalar_type() == at::kLong && slot->is_contiguous() && slot->numel() == T, "latent_prep: pages [blocks, block_size, kv_rank + rot]");
    ps = pages->stride(0); bs = (int)pages->size(1); slots = pages->size(0) * pages->size(1);
  }
  verl_count_launches(1);
  CHECK_RC(vb_latent_prep(dt, p.data_ptr(), p.stride(0), ptr(qn), kn.data_ptr(), (float)eps, pos.data_ptr<int>(), cs.data_ptr<float>(),
                          sn.data_ptr<float>(), (int)(2 * cs.size(1)), (int)cs.size(0), cq.data_ptr(), want_rows ? lat.data_ptr() : nullptr, kr + rot, ptr(pages), ps, bs,
                          slots, pages.has_value() ? lptr(*slot) : nullptr, (int)T, (int)qr, (int)kr, (int)rot, cur_stream()), "vb_latent_prep");
  return {cq, lat};
}

Tensor gather_pages(const Tensor& pages, const Tensor& block_table, const Tensor& cu_k, const Tensor& k_start, int64_t total) {
  const int dt = dtype_of(pages);
  CHECK_I32(block_table);
  CHECK_I32(cu_k);
  CHECK_I32(k_start);
  const c10::cuda::CUDAGuard guard(pages.device());
  Tensor out = at::empty({total, pages.size(2)}, pages.options());
  verl_count_launches(1);
  CHECK_RC(vb_gather_pages(dt, pages.data_ptr(), pages.stride(0), (int)pages.size(1), block_table.data_ptr<int>(), (int)block_table.size(1), cu_k.data_ptr<int>(),
                           k_start.data_ptr<int>(), (int)k_start.numel(), (int)pages.size(2), out.data_ptr(), (int)total, cur_stream()), "vb_gather_pages");
  return out;
}

// out[m, h, :] = a[m, h, :] w[h] (b_mn: w [H, K, N]) or a[m, h, :] w[h]^T (w [H, N, K]), times sigmoid(gate[m, h]), into out with
// the given strides; tensor cores where the sizes allow.
void run_headwise(const Tensor& a, const Tensor& w, bool b_mn, const OptTensor& gate, VbHeadwise p) {
  const int dt = dtype_of(a);
  same(a, w, "headwise_linear");
  TORCH_CHECK(a.dim() == 3 && w.dim() == 3 && a.size(1) == w.size(0) && a.stride(2) == 1 && w.stride(2) == 1, "headwise_linear");
  p.a = a.data_ptr(); p.lda = a.stride(0); p.a_head = a.stride(1);
  p.w = w.data_ptr(); p.w_head = w.stride(0); p.ldw = w.stride(1); p.kn = b_mn;
  p.M = (int)a.size(0); p.H = (int)a.size(1); p.K = (int)(b_mn ? w.size(1) : w.size(2)); p.N = (int)(b_mn ? w.size(2) : w.size(1));
  if (gate.has_value()) {
    CHECK_F32(*gate);
    TORCH_CHECK(gate->size(0) == p.M && gate->size(1) >= p.H && gate->stride(1) == 1, "headwise_linear: gate [M, H]");
    p.gate = gate->data_ptr<float>(); p.ldg = gate->stride(0);
  }
  verl_count_launches(1);
  int rc = dt == 1 ? vb_headwise(&p, cur_stream()) : -1;
  if (rc < 0) {
    VbEpiArgs e{};
    e.mode = VB_EPI_STORE;
    e.D = p.out; e.ldd = p.ldo; e.gate = p.gate; e.ldg = p.ldg;
    rc = vb_gemm_simt(dt, p.a, p.w, p.M, p.N, p.K, p.lda, p.ldw, b_mn, p.H, p.a_head, p.w_head, p.o_head, &e, cur_stream());
    if (rc == 0 && p.rot > 0) {
      verl_count_launches(1);
      rc = vb_rope_copy(dt, p.a, p.lda, (int)p.a_head, p.K, p.out, p.ldo, (int)p.o_head, p.N, p.pos, p.cos_t, p.sin_t, p.M, p.H, p.rot, p.half, p.max_pos, cur_stream());
    }
  }
  CHECK_RC(rc, "headwise_linear");
}

Tensor headwise_linear(const Tensor& a, const Tensor& w, bool b_mn, const OptTensor& gate) {
  TORCH_CHECK(a.dim() == 3 && w.dim() == 3 && a.size(2) == (b_mn ? w.size(1) : w.size(2)), "headwise_linear: sizes");
  const c10::cuda::CUDAGuard guard(a.device());
  const int64_t N = b_mn ? w.size(2) : w.size(1);
  Tensor d = at::empty({a.size(0), a.size(1), N}, a.options());
  VbHeadwise p{};
  p.out = d.data_ptr(); p.ldo = d.stride(0); p.o_head = N;
  run_headwise(a, w, b_mn, gate, p);
  return d;
}

// q [S, H, dim + rot], uk [H, dim, rank]: [q_unrotated uk | rotated part] as [S, H, rank + rot].
Tensor latent_absorb(const Tensor& q, const Tensor& uk, const Tensor& pos, const Tensor& cs, const Tensor& sn) {
  CHECK_I32(pos);
  CHECK_F32(cs);
  const int64_t rot = q.size(2) - uk.size(1), rank = uk.size(2);
  TORCH_CHECK(q.dim() == 3 && rot >= 0 && 2 * cs.size(1) <= rot && cs.is_contiguous() && sn.is_contiguous() && pos.numel() == q.size(0), "latent_absorb: sizes");
  const c10::cuda::CUDAGuard guard(q.device());
  Tensor out = at::empty({q.size(0), q.size(1), rank + rot}, q.options());
  VbHeadwise p{};
  p.out = out.data_ptr(); p.ldo = out.stride(0); p.o_head = rank + rot;
  p.rot = (int)rot; p.half = (int)cs.size(1); p.max_pos = (int)cs.size(0); p.pos = pos.data_ptr<int>(); p.cos_t = cs.data_ptr<float>(); p.sin_t = sn.data_ptr<float>();
  run_headwise(q, uk, true, OptTensor(), p);
  return out;
}

// Prompt attention: q [T, H, du + dr], ku [Tk, H, du], kr [Tk, dr], v [Tk, H, dv] (strided views), cu_q / cu_k int32 [B + 1].
Tensor latent_attn_prefill(const Tensor& q, const Tensor& ku, const Tensor& kr, const Tensor& v, const Tensor& cu_q, const Tensor& cu_k,
                           const OptTensor& sink, const OptTensor& gate, int64_t window, double scale, int64_t keep_first) {
  const int dt = dtype_of(q);
  CHECK_I32(cu_q);
  CHECK_I32(cu_k);
  same(q, ku, "latent_attn_prefill");
  TORCH_CHECK(q.dim() == 3 && ku.dim() == 3 && kr.dim() == 2 && v.dim() == 3 && q.stride(2) == 1 && ku.stride(2) == 1 && kr.stride(1) == 1 && v.stride(2) == 1 &&
              q.size(2) == ku.size(2) + kr.size(1) && ku.size(1) == q.size(1) && v.size(1) == q.size(1) && cu_q.numel() == cu_k.numel(), "latent_attn_prefill");
  const c10::cuda::CUDAGuard guard(q.device());
  VbLatentAttn a{};
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.hq = (int)q.stride(1);
  a.ku = ku.data_ptr(); a.ku_row = ku.stride(0); a.ku_head = (int)ku.stride(1);
  a.kr = kr.data_ptr(); a.kr_row = kr.stride(0);
  a.v = v.data_ptr(); a.v_row = v.stride(0); a.v_head = (int)v.stride(1);
  a.cu_q = cu_q.data_ptr<int>(); a.cu_k = cu_k.data_ptr<int>();
  a.T = (int)q.size(0); a.H = (int)q.size(1); a.du = (int)ku.size(2); a.dr = (int)kr.size(1); a.dv = (int)v.size(2);
  a.B = (int)cu_q.numel() - 1; a.window = (int)window; a.keep_first = (int)keep_first; a.scale = (float)scale;
  if (sink.has_value()) { same(q, *sink, "latent_attn_prefill"); TORCH_CHECK(sink->numel() == a.H); a.sink = sink->data_ptr(); }
  if (gate.has_value()) { CHECK_F32(*gate); TORCH_CHECK(gate->size(0) == a.T && gate->stride(1) == 1); a.gate = gate->data_ptr<float>(); a.ldg = gate->stride(0); }
  Tensor out = at::empty({q.size(0), q.size(1), v.size(2)}, q.options());
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  verl_count_launches(1);
  int rc = dt == 1 && a.T > 0 ? vb_latent_prefill(&a, (int)ku.size(0), cur_stream()) : -1;
  if (rc < 0) rc = vb_latent_attn_simt(dt, &a, 0, cur_stream());
  CHECK_RC(rc, "latent_attn_prefill");
  return out;
}

// Decode attention in the latent space: q [S, H, kv_rank + rot] (absorbed query, rotated part last), pages [blocks, block_size, kv_rank + rot].
Tensor latent_attn_decode(const Tensor& q, const Tensor& pages, const Tensor& block_table, const Tensor& ctx_len, const OptTensor& sink,
                          int64_t kv_rank, int64_t window, double scale, int64_t keep_first) {
  const int dt = dtype_of(q);
  same(q, pages, "latent_attn_decode");
  CHECK_I32(block_table);
  CHECK_I32(ctx_len);
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && pages.dim() == 3 && pages.stride(2) == 1 && pages.size(2) == q.size(2) && kv_rank > 0 && kv_rank <= q.size(2) &&
              block_table.size(0) == q.size(0) && ctx_len.numel() == q.size(0), "latent_attn_decode");
  const c10::cuda::CUDAGuard guard(q.device());
  VbLatentAttn a{};
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.hq = (int)q.stride(1);
  char* base = reinterpret_cast<char*>(pages.data_ptr());
  a.ku = base; a.ku_row = pages.stride(1);
  a.kr = base + kv_rank * pages.element_size(); a.kr_row = pages.stride(1);
  a.v = base; a.v_row = pages.stride(1);
  a.block_table = block_table.data_ptr<int>(); a.max_blocks = (int)block_table.size(1); a.block_size = (int)pages.size(1); a.page_stride = pages.stride(0);
  a.ctx_len = ctx_len.data_ptr<int>();
  a.T = a.B = (int)q.size(0); a.H = (int)q.size(1); a.du = (int)kv_rank; a.dr = (int)(q.size(2) - kv_rank); a.dv = (int)kv_rank;
  a.window = (int)window; a.keep_first = (int)keep_first; a.scale = (float)scale;
  if (sink.has_value()) { same(q, *sink, "latent_attn_decode"); TORCH_CHECK(sink->numel() == a.H); a.sink = sink->data_ptr(); }
  Tensor out = at::empty({q.size(0), q.size(1), kv_rank}, q.options());
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  if (dt == 1) {
    const int64_t all = (int64_t)a.max_blocks * a.block_size;
    const int ns = vb_latent_decode_splits(a.B, a.H, a.dv, a.du + a.dr, a.block_size, (int)(window > 0 ? std::min<int64_t>(window + keep_first + 64, all) : all));
    if (ns > 0) {
      Tensor po, ml;
      if (ns > 1) {
        po = at::empty({a.B, a.H, ns, kv_rank}, q.options().dtype(at::kFloat));
        ml = at::empty({a.B, a.H, ns, 2}, q.options().dtype(at::kFloat));
      }
      const int rc = vb_latent_decode(&a, pages.size(0), ns, ns > 1 ? po.data_ptr<float>() : nullptr, ns > 1 ? ml.data_ptr<float>() : nullptr, cur_stream());
      if (rc >= 0) {
        verl_count_launches(ns > 1 ? 2 : 1);
        CHECK_RC(rc, "vb_latent_decode");
        return out;
      }
    }
  }
  verl_count_launches(1);
  CHECK_RC(vb_latent_attn_simt(dt, &a, 0, cur_stream()), "vb_latent_attn_simt");
  return out;
}

// ---- stacks with RMS norms on the sublayer outputs
std::tuple<Tensor, Tensor> embed_rms(const Tensor& ids, const Tensor& w, double scale, const Tensor& nw, double eps) {
  const int dt = dtype_of(w);
  const c10::cuda::CUDAGuard guard(w.device());
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous() && w.dim() == 2 && w.is_contiguous() && nw.numel() == w.size(1), "embed_rms");
  same(w, nw, "embed_rms");
  const int T = (int)ids.numel(), W = (int)w.size(1);
  Tensor x = at::empty({T, W}, w.options().dtype(at::kFloat)), h = at::empty({T, W}, w.options());
  verl_count_launches(1);
  CHECK_RC(vb_embed_rms(dt, lptr(ids), w.data_ptr(), (float)scale, nw.data_ptr(), (float)eps, x.data_ptr<float>(), h.data_ptr(), T, W, (int)w.size(0), cur_stream()),
           "vb_embed_rms");
  return {x, h};
}

// a w^T for a row kernel: fp32 partial products [splits, M, N] where the GEMM splits K, else [M, N] in a's type.
Tensor linear_partial(const Tensor& a, const Tensor& w) {
  const c10::cuda::CUDAGuard guard(a.device());
  const int dt = dtype_of(a);
  same(a, w, "linear_partial");
  TORCH_CHECK(a.dim() == 2 && w.dim() == 2 && a.stride(1) == 1 && w.stride(1) == 1 && a.size(1) == w.size(1), "linear_partial: a [M, K], w [N, K]");
  const int M = (int)a.size(0), K = (int)a.size(1), N = (int)w.size(0);
  if (dt == 1 && M > 0 && M <= 1024 && N % 8 == 0 && K % 8 == 0 && a.stride(0) % 8 == 0 && w.stride(0) % 8 == 0) {
    const int s = vb_gemm_skinny_splits(M, N, K);
    if (s > 1) {
      Tensor ws = at::empty({s, M, N}, a.options().dtype(at::kFloat));
      const int rc = vb_gemm_skinny(a.data_ptr(), w.data_ptr(), nullptr, nullptr, M, N, K, a.stride(0), w.stride(0), 0, s, ws.data_ptr<float>(), 0, 1, cur_stream());
      if (rc == 0) {
        verl_count_launches(1);
        return ws;
      }
      TORCH_CHECK(rc < 0, "linear_partial failed with code ", rc);
    }
  }
  return linear_act(a, w, false, false);
}

Tensor linear_softcap(const Tensor& a, const Tensor& w, double cap) {
  const c10::cuda::CUDAGuard guard(a.device());
  TORCH_CHECK(cap > 0, "linear_softcap: cap > 0");
  Tensor d = at::empty({a.size(0), w.size(0)}, a.options());
  VbEpiArgs e{};
  e.mode = VB_EPI_SOFTCAP;
  e.cap = (float)cap;
  e.D = d.data_ptr(); e.ldd = d.stride(0);
  run_gemm(a, w, e);
  return d;
}

// x += mult * rms_norm(Y) nw (see VbResidRms); returns the new stream, or its norm with `next`, in nw's type.
Tensor residual_rms_(Tensor x, const OptTensor& y, const Tensor& nw, double eps, double mult, const OptTensor& next, const OptTensor& rows, const OptTensor& slot,
                     const OptTensor& gate) {
  CHECK_F32(x);
  const int dt = dtype_of(nw);
  const c10::cuda::CUDAGuard guard(x.device());
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && nw.numel() == x.size(1) && (y.has_value() || rows.has_value()), "residual_rms_: x [T, W]");
  VbResidRms p{};
  p.T = (int)x.size(0); p.W = (int)x.size(1);
  p.x = x.data_ptr<float>(); p.nw = nw.data_ptr(); p.eps = (float)eps; p.mult = (float)mult;
  if (y.has_value()) {
    const bool parts = y->dim() == 3;
    TORCH_CHECK(y->is_cuda() && y->size(-1) == p.W && y->size(-2) == p.T && y->stride(-1) == 1, "residual_rms_: y");
    if (parts) { CHECK_F32(*y); } else { same(nw, *y, "residual_rms_"); }
    p.y = y->data_ptr(); p.y_f32 = parts; p.splits = parts ? (int)y->size(0) : 1; p.split_stride = parts ? y->stride(0) : 0; p.ldy = y->stride(-2);
  }
  if (rows.has_value()) {
    same(nw, *rows, "residual_rms_");
    TORCH_CHECK(slot.has_value() && rows->dim() == 2 && rows->size(1) == p.W && rows->stride(1) == 1 && slot->dim() == 2 && slot->size(0) == p.T, "residual_rms_: rows");
    CHECK_I32(*slot);
    p.rows = rows->data_ptr(); p.ldr = rows->stride(0); p.slot = slot->data_ptr<int>(); p.top = (int)slot->size(1);
  }
  if (gate.has_value()) {
    CHECK_F32(*gate);
    TORCH_CHECK(gate->dim() == 1 && gate->numel() == p.T, "residual_rms_: gate [T]");
    p.gate = gate->data_ptr<float>(); p.ldgate = gate->stride(0);
  }
  if (next.has_value()) { same(nw, *next, "residual_rms_"); TORCH_CHECK(next->numel() == p.W); p.next = next->data_ptr(); }
  Tensor h = at::empty({p.T, p.W}, nw.options());
  p.h = h.data_ptr();
  verl_count_launches(1);
  CHECK_RC(vb_residual_rms(dt, &p, cur_stream()), "vb_residual_rms");
  return h;
}

Tensor gated_silu_rows(const Tensor& gu, const float* row_scale, float clip) {
  const int dt = dtype_of(gu);
  TORCH_CHECK(gu.dim() == 2 && gu.stride(1) == 1 && gu.size(1) % 2 == 0, "gated_silu: [T, 2 I]");
  Tensor out = at::empty({gu.size(0), gu.size(1) / 2}, gu.options());
  verl_count_launches(1);
  CHECK_RC(vb_gated_silu(dt, gu.data_ptr(), gu.stride(0), row_scale, clip, out.data_ptr(), (int)out.size(0), (int)out.size(1), cur_stream()), "vb_gated_silu");
  return out;
}
Tensor gated_silu(const Tensor& gu) {
  const c10::cuda::CUDAGuard guard(gu.device());
  return gated_silu_rows(gu, nullptr, 0.f);
}

// Router and expert-grouped copies of the tokens: (x [rows, W], slot [T, k], score per row, expert per 128-row tile, number of tiles).
std::tuple<Tensor, Tensor, Tensor, Tensor, Tensor> expert_dispatch(const Tensor& h, const Tensor& z, int64_t E, int64_t k, bool renorm,
                                                                   const OptTensor& corr, int64_t groups, int64_t keep) {
  const int dt = dtype_of(h);
  CHECK_F32(z);
  const c10::cuda::CUDAGuard guard(h.device());
  const int64_t T = h.size(0), W = h.size(1);
  TORCH_CHECK(h.dim() == 2 && h.stride(1) == 1 && z.dim() == 2 && z.stride(1) == 1 && z.size(0) == T && z.size(1) >= E && k >= 1 && k <= E, "expert_dispatch");
  TORCH_CHECK(groups >= 1 && E % groups == 0 && keep >= 1 && keep <= groups && k <= keep * (E / groups), "expert_dispatch: groups");
  if (corr.has_value()) { same(h, *corr, "expert_dispatch"); TORCH_CHECK(corr->numel() == E && corr->is_contiguous(), "expert_dispatch: correction [E]"); }
  const int64_t tiles = std::max<int64_t>(1, (T * k + 127) / 128 + std::min<int64_t>(E, T * k));
  const auto i32 = h.options().dtype(at::kInt), f32 = h.options().dtype(at::kFloat);
  Tensor counts = at::zeros({E}, i32), expert = at::empty({T, k}, i32), rank = at::empty({T, k}, i32), slot = at::empty({T, k}, i32);
  Tensor score = at::empty({T, k}, f32), row_scale = at::empty({tiles * 128}, f32), tile_expert = at::empty({tiles}, i32), num_tiles = at::empty({1}, i32);
  Tensor x = at::empty({tiles * 128, W}, h.options());
  if (T == 0) { num_tiles.zero_(); return {x, slot, row_scale, tile_expert, num_tiles}; }
  verl_count_launches(2);
  CHECK_RC(vb_expert_route(dt, z.data_ptr<float>(), z.stride(0), ptr(corr), (int)groups, (int)keep, (int)T, (int)E, (int)k, renorm, score.data_ptr<float>(), expert.data_ptr<int>(), rank.data_ptr<int>(),
                           counts.data_ptr<int>(), cur_stream()), "vb_expert_route");
  CHECK_RC(vb_expert_place(dt, h.data_ptr(), h.stride(0), score.data_ptr<float>(), expert.data_ptr<int>(), rank.data_ptr<int>(), counts.data_ptr<int>(), (int)T, (int)E,
                           (int)k, (int)W, x.data_ptr(), row_scale.data_ptr<float>(), slot.data_ptr<int>(), tile_expert.data_ptr<int>(), num_tiles.data_ptr<int>(),
                           (int)tiles, cur_stream()), "vb_expert_place");
  return {x, slot, row_scale, tile_expert, num_tiles};
}

// out[rows, N] = a w_e^T per 128-row tile, w [E, N, K]: tensor cores where the sizes allow.
Tensor expert_linear(const Tensor& a, const Tensor& w, const Tensor& tile_expert, const Tensor& num_tiles) {
  const int dt = dtype_of(a);
  same(a, w, "expert_linear");
  CHECK_I32(tile_expert);
  CHECK_I32(num_tiles);
  TORCH_CHECK(a.dim() == 2 && a.stride(1) == 1 && a.size(0) == tile_expert.numel() * 128 && w.dim() == 3 && w.is_contiguous() && w.size(2) == a.size(1), "expert_linear");
  const c10::cuda::CUDAGuard guard(a.device());
  const int rows = (int)a.size(0), N = (int)w.size(1), K = (int)w.size(2), E = (int)w.size(0);
  Tensor d = at::empty({rows, N}, a.options());
  verl_count_launches(1);
  int rc = -1;
  if (dt == 1 && K % 8 == 0)
    rc = vb_gemm_grouped(1, a.data_ptr(), w.data_ptr(), d.data_ptr(), rows, rows, N, K, a.stride(0), K, N, 0, 0, E, tile_expert.data_ptr<int>(),
                         num_tiles.data_ptr<int>(), nullptr, cur_stream());
  if (rc < 0) {
    VbEpiArgs e{};
    e.mode = VB_EPI_STORE;
    e.D = d.data_ptr(); e.ldd = N;
    rc = vb_gemm_simt_grouped(dt, a.data_ptr(), w.data_ptr(), rows, N, K, a.stride(0), tile_expert.data_ptr<int>(), num_tiles.data_ptr<int>(), &e, cur_stream());
  }
  CHECK_RC(rc, "expert_linear");
  return d;
}

// act[rows, I] = silu(s g) * (s u), [g | u] = x w_e^T, w [E, 2 I, K], s = scale[row]; clip > 0: s g sigmoid(1.702 g) (u + 1), g <= clip, |u| <= clip.
Tensor expert_up(const Tensor& x, const Tensor& w, const Tensor& scale, const Tensor& tile_expert, const Tensor& num_tiles, double clip) {
  CHECK_F32(scale);
  CHECK_I32(tile_expert);
  CHECK_I32(num_tiles);
  same(x, w, "expert_up");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && scale.numel() == x.size(0) && x.size(0) == tile_expert.numel() * 128 && w.dim() == 3 && w.is_contiguous() &&
              w.size(2) == x.size(1) && w.size(1) % 2 == 0, "expert_up");
  const c10::cuda::CUDAGuard guard(x.device());
  const int rows = (int)x.size(0), I = (int)w.size(1) / 2, K = (int)w.size(2);
  if (dtype_of(x) == 1) {
    Tensor act = at::empty({rows, I}, x.options());
    const int rc = vb_gemm_grouped_swiglu(x.data_ptr(), w.data_ptr(), act.data_ptr(), rows, I, K, x.stride(0), I, scale.data_ptr<float>(), (int)w.size(0),
                                          tile_expert.data_ptr<int>(), num_tiles.data_ptr<int>(), (float)clip, cur_stream());
    if (rc >= 0) {
      verl_count_launches(1);
      CHECK_RC(rc, "expert_up");
      return act;
    }
  }
  return gated_silu_rows(expert_linear(x, w, tile_expert, num_tiles), scale.data_ptr<float>(), (float)clip);
}

// p [T, q | k | v]; see VbQkvPrep. Returns (queries [T, H, dim], rows [T or 0, G (dim + vdim)]).
std::tuple<Tensor, Tensor> qkv_prep(const Tensor& p, const Tensor& qn, const Tensor& kn, double eps, const Tensor& pos, const Tensor& cs, const Tensor& sn, int64_t H,
                                    int64_t G, int64_t vdim, const OptTensor& vfirst, const OptTensor& vmix, const OptTensor& pages, const OptTensor& slot,
                                    bool want_rows) {
  const int dt = dtype_of(p);
  CHECK_I32(pos);
  CHECK_F32(cs);
  CHECK_F32(sn);
  same(p, qn, "qkv_prep");
  same(p, kn, "qkv_prep");
  const int64_t T = p.size(0), dim = qn.numel(), width = G * (dim + vdim);
  TORCH_CHECK(p.dim() == 2 && p.stride(1) == 1 && p.size(1) >= (H + G) * dim + G * vdim && kn.numel() == dim && pos.numel() == T && cs.is_contiguous() &&
              sn.is_contiguous() && cs.dim() == 2 && 2 * cs.size(1) <= dim, "qkv_prep: sizes");
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor q = at::empty({T, H, dim}, p.options()), rows = at::empty({want_rows ? T : 0, width}, p.options());
  VbQkvPrep a{};
  a.p = p.data_ptr(); a.ldp = p.stride(0); a.qn = qn.data_ptr(); a.kn = kn.data_ptr(); a.pos = pos.data_ptr<int>();
  a.cos_t = cs.data_ptr<float>(); a.sin_t = sn.data_ptr<float>(); a.half = (int)cs.size(1); a.max_pos = (int)cs.size(0);
  if (vfirst.has_value()) {
    same(p, *vfirst, "qkv_prep");
    TORCH_CHECK(vmix.has_value() && vmix->numel() == 1 && vfirst->dim() == 2 && vfirst->size(0) == T && vfirst->size(1) == G * vdim && vfirst->stride(1) == 1, "qkv_prep: v_first");
    same(p, *vmix, "qkv_prep");
    a.vfirst = vfirst->data_ptr(); a.ldvf = vfirst->stride(0); a.vmix = vmix->data_ptr();
  }
  a.q = q.data_ptr();
  a.ldr = width;
  if (want_rows) a.rows = rows.data_ptr();
  a.block_size = 1;
  if (pages.has_value()) {
    same(p, *pages, "qkv_prep");
    TORCH_CHECK(pages->dim() == 3 && pages->size(2) == width && pages->stride(2) == 1 && pages->stride(1) == width && slot.has_value() && slot->is_cuda() &&
                slot->scalar_type() == at::kLong && slot->is_contiguous() && slot->numel() == T, "qkv_prep: pages [blocks, block_size, kv_heads (dim + vdim)]");
    a.pages = pages->data_ptr(); a.page_stride = pages->stride(0); a.block_size = (int)pages->size(1); a.num_slots = pages->size(0) * pages->size(1); a.slot = lptr(*slot);
  }
  a.T = (int)T; a.H = (int)H; a.G = (int)G; a.dim = (int)dim; a.vdim = (int)vdim; a.eps = (float)eps;
  verl_count_launches(1);
  CHECK_RC(vb_qkv_prep(dt, &a, cur_stream()), "vb_qkv_prep");
  return {q, rows};
}

// Differential attention over q [*, 2 H, d]: arguments of the difference; `out` [T, H, e].
void diff_args(VbLatentAttn& a, const Tensor& q, const OptTensor& vec, double diff, double eps) {
  a.maps = vec.has_value() ? 2 : 1;
  if (!vec.has_value()) return;
  same(q, *vec, "differential attention");
  TORCH_CHECK(q.size(1) % 2 == 0 && vec->is_contiguous() && vec->numel() == 4 * q.size(2), "differential attention: four vectors of a map's size");
  a.diff_vec = vec->data_ptr(); a.diff = (float)diff; a.eps = (float)eps;
}
// The difference behind an attention kernel that leaves the maps apart.
void diff_simt(int dt, VbLatentAttn a, const Tensor& q, const Tensor& out) {
  Tensor maps = at::empty({a.T, a.H, a.dv}, q.options().dtype(at::kFloat));
  a.out = maps.data_ptr(); a.ldo = maps.stride(0);
  verl_count_launches(2);
  CHECK_RC(vb_latent_attn_simt(dt, &a, 1, cur_stream()), "vb_latent_attn_simt");
  CHECK_RC(vb_diff_combine(dt, maps.data_ptr(), 1, a.diff_vec, a.du, a.diff, a.eps, out.data_ptr(), a.T, a.H / 2, a.dv, cur_stream()), "vb_diff_combine");
}

// Prompt attention: q [T, H, d], k [Tk, G, d], v [Tk, G, e] (strided views), cu_q / cu_k int32 [B + 1]; with `vec` q [T, 2 H, d], k [Tk, 2 G, d].
Tensor grouped_attn_prefill(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& cu_q, const Tensor& cu_k, const OptTensor& sink, int64_t window,
                            double scale, double softcap, int64_t keep_first, int64_t chunk, const OptTensor& vec, double diff, double eps) {
  const int dt = dtype_of(q);
  CHECK_I32(cu_q);
  CHECK_I32(cu_k);
  same(q, k, "grouped_attn_prefill");
  same(q, v, "grouped_attn_prefill");
  TORCH_CHECK(q.dim() == 3 && k.dim() == 3 && v.dim() == 3 && q.stride(2) == 1 && k.stride(2) == 1 && v.stride(2) == 1 && q.size(2) == k.size(2) && k.size(1) > 0 &&
              q.size(1) % k.size(1) == 0 && v.size(1) * (vec.has_value() ? 2 : 1) == k.size(1) && v.size(0) == k.size(0) && cu_q.numel() == cu_k.numel() &&
              !(chunk > 0 && window > 0), "grouped_attn_prefill");
  const c10::cuda::CUDAGuard guard(q.device());
  VbLatentAttn a{};
  diff_args(a, q, vec, diff, eps);
  a.chunk = (int)chunk;
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.hq = (int)q.stride(1);
  a.ku = k.data_ptr(); a.ku_row = k.stride(0); a.ku_head = (int)k.stride(1);
  a.v = v.data_ptr(); a.v_row = v.stride(0); a.v_head = (int)v.stride(1);
  a.cu_q = cu_q.data_ptr<int>(); a.cu_k = cu_k.data_ptr<int>();
  a.T = (int)q.size(0); a.H = (int)q.size(1); a.du = (int)q.size(2); a.dv = (int)v.size(2); a.B = (int)cu_q.numel() - 1;
  a.window = (int)window; a.keep_first = (int)keep_first; a.scale = (float)scale; a.softcap = (float)softcap; a.kv_group = (int)(q.size(1) / k.size(1));   // query heads per key / value head, maps not counted
  if (sink.has_value()) { same(q, *sink, "grouped_attn_prefill"); TORCH_CHECK(sink->numel() == a.H); a.sink = sink->data_ptr(); }
  Tensor out = at::empty({q.size(0), q.size(1) / a.maps, v.size(2)}, q.options());
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  int rc = dt == 1 && a.T > 0 ? vb_latent_prefill(&a, (int)k.size(0), cur_stream()) : -1;
  if (rc >= 0) verl_count_launches(1);
  if (rc < 0 && a.maps > 1) {
    // values too wide for both maps' products at once: the maps as heads of their own over the values of their pair
    if (dt == 1 && a.T > 0) {
      VbLatentAttn m = a;
      Tensor both = at::empty({a.T, a.H, a.dv}, q.options());
      m.maps = 1; m.kv_group = a.kv_group; m.split_maps = 1; m.out = both.data_ptr(); m.ldo = both.stride(0);
      rc = vb_latent_prefill(&m, (int)k.size(0), cur_stream());
      if (rc == 0) {
        verl_count_launches(2);
        CHECK_RC(vb_diff_combine(dt, both.data_ptr(), 0, a.diff_vec, a.du, a.diff, a.eps, out.data_ptr(), a.T, a.H / 2, a.dv, cur_stream()), "vb_diff_combine");
        return out;
      }
    }
    if (rc < 0) {
      diff_simt(dt, a, q, out);
      return out;
    }
  }
  if (rc < 0) verl_count_launches(1);
  if (rc < 0) rc = vb_latent_attn_simt(dt, &a, 0, cur_stream());
  CHECK_RC(rc, "grouped_attn_prefill");
  return out;
}

// Decode attention: q [S, H, d], pages [blocks, block_size, G (d + vdim)] with rows [keys | values].
Tensor grouped_attn_decode(const Tensor& q, const Tensor& pages, const Tensor& block_table, const Tensor& ctx_len, const OptTensor& sink, int64_t G, int64_t vdim,
                           int64_t window, double scale, double softcap, int64_t keep_first, int64_t chunk, const OptTensor& vec, double diff, double eps) {
  const int dt = dtype_of(q);
  const int64_t maps = vec.has_value() ? 2 : 1;
  same(q, pages, "grouped_attn_decode");
  CHECK_I32(block_table);
  CHECK_I32(ctx_len);
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && pages.dim() == 3 && pages.stride(2) == 1 && G > 0 && q.size(1) % (G * maps) == 0 &&
              pages.size(2) == G * (maps * q.size(2) + vdim) && block_table.size(0) == q.size(0) && ctx_len.numel() == q.size(0) && !(chunk > 0 && window > 0), "grouped_attn_decode");
  const c10::cuda::CUDAGuard guard(q.device());
  VbLatentAttn a{};
  diff_args(a, q, vec, diff, eps);
  a.chunk = (int)chunk;
  const int64_t d = q.size(2);
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.hq = (int)q.stride(1);
  char* base = reinterpret_cast<char*>(pages.data_ptr());
  a.ku = base; a.ku_row = pages.stride(1); a.ku_head = (int)d;
  a.kr = base;
  a.v = base + G * maps * d * pages.element_size(); a.v_row = pages.stride(1); a.v_head = (int)vdim;
  a.block_table = block_table.data_ptr<int>(); a.max_blocks = (int)block_table.size(1); a.block_size = (int)pages.size(1); a.page_stride = pages.stride(0);
  a.ctx_len = ctx_len.data_ptr<int>();
  a.T = a.B = (int)q.size(0); a.H = (int)q.size(1); a.du = (int)d; a.dv = (int)vdim;
  a.window = (int)window; a.keep_first = (int)keep_first; a.scale = (float)scale; a.softcap = (float)softcap; a.kv_group = (int)(q.size(1) / (G * maps));
  if (sink.has_value()) { same(q, *sink, "grouped_attn_decode"); TORCH_CHECK(sink->numel() == a.H); a.sink = sink->data_ptr(); }
  Tensor out = at::empty({q.size(0), q.size(1) / maps, vdim}, q.options());
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  if (dt == 1) {
    const int64_t all = (int64_t)a.max_blocks * a.block_size;
    const int ns = vb_grouped_decode_splits(&a, (int)(window > 0 ? std::min<int64_t>(window + keep_first + 128, all) : chunk > 0 ? std::min<int64_t>(chunk + 64, all) : all));
    if (ns > 0) {
      Tensor po, ml;
      if (ns > 1) {
        po = at::empty({a.B, a.H, ns, vdim}, q.options().dtype(at::kFloat));
        ml = at::empty({a.B, a.H, ns, 2}, q.options().dtype(at::kFloat));
      }
      const int rc = vb_grouped_decode(&a, pages.size(0), ns, ns > 1 ? po.data_ptr<float>() : nullptr, ns > 1 ? ml.data_ptr<float>() : nullptr, cur_stream());
      if (rc >= 0) {
        verl_count_launches(ns > 1 ? 2 : 1);
        CHECK_RC(rc, "vb_grouped_decode");
        return out;
      }
    }
  }
  if (maps > 1) {
    diff_simt(dt, a, q, out);
    return out;
  }
  verl_count_launches(1);
  CHECK_RC(vb_latent_attn_simt(dt, &a, 0, cur_stream()), "vb_latent_attn_simt");
  return out;
}

// p [T, q | k | v]; see VbWholeNorm. Returns (queries [T, H, dim], rows [T or 0, G (dim + vdim)]).
std::tuple<Tensor, Tensor> whole_norm_prep(const Tensor& p, const Tensor& qn, const Tensor& kn, const Tensor& temp, double eps, int64_t H, int64_t G, int64_t vdim,
                                           const OptTensor& pages, const OptTensor& slot, bool want_rows) {
  const int dt = dtype_of(p);
  for (const Tensor* t : {&qn, &kn, &temp}) same(p, *t, "whole_norm_prep");
  const int64_t T = p.size(0), dim = qn.numel() / H, width = G * (dim + vdim);
  TORCH_CHECK(p.dim() == 2 && p.stride(1) == 1 && qn.numel() == H * dim && kn.numel() == G * dim && temp.numel() == H && p.size(1) >= (H + G) * dim + G * vdim, "whole_norm_prep: sizes");
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor q = at::empty({T, H, dim}, p.options()), rows = at::empty({want_rows ? T : 0, width}, p.options());
  VbWholeNorm a{};
  a.p = p.data_ptr(); a.ldp = p.stride(0); a.qn = qn.data_ptr(); a.kn = kn.data_ptr(); a.temp = temp.data_ptr(); a.q = q.data_ptr(); a.ldr = width;
  if (want_rows) a.rows = rows.data_ptr();
  a.block_size = 1;
  if (pages.has_value()) {
    same(p, *pages, "whole_norm_prep");
    TORCH_CHECK(pages->dim() == 3 && pages->size(2) == width && pages->stride(2) == 1 && pages->stride(1) == width && slot.has_value() && slot->is_cuda() &&
                slot->scalar_type() == at::kLong && slot->is_contiguous() && slot->numel() == T, "whole_norm_prep: pages [blocks, block_size, kv_heads (dim + vdim)]");
    a.pages = pages->data_ptr(); a.page_stride = pages->stride(0); a.block_size = (int)pages->size(1); a.num_slots = pages->size(0) * pages->size(1); a.page_slot = lptr(*slot);
  }
  a.T = (int)T; a.H = (int)H; a.G = (int)G; a.dim = (int)dim; a.vdim = (int)vdim; a.eps = (float)eps;
  verl_count_launches(1);
  CHECK_RC(vb_whole_norm(dt, &a, cur_stream()), "vb_whole_norm");
  return {q, rows};
}

Tensor embed_rows(const Tensor& ids, const Tensor& w, double scale) {
  const int dt = dtype_of(w);
  const c10::cuda::CUDAGuard guard(w.device());
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous() && w.dim() == 2 && w.is_contiguous(), "embed_rows");
  Tensor x = at::empty({ids.numel(), w.size(1)}, w.options().dtype(at::kFloat));
  verl_count_launches(1);
  CHECK_RC(vb_embed_rows(dt, lptr(ids), w.data_ptr(), (float)scale, x.data_ptr<float>(), (int)ids.numel(), (int)w.size(1), (int)w.size(0), cur_stream()), "vb_embed_rows");
  return x;
}

// See VbRmsConv: cu given: portions, else one token per row.
Tensor rms_conv(Tensor x, const OptTensor& y, const OptTensor& bias, const Tensor& nw, double eps, const OptTensor& conv, const OptTensor& cu, const OptTensor& state,
                const OptTensor& slots, const OptTensor& fresh, const OptTensor& active) {
  CHECK_F32(x);
  const int dt = dtype_of(nw);
  const c10::cuda::CUDAGuard guard(x.device());
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && nw.numel() == x.size(1) && nw.is_contiguous(), "rms_conv: x [T, W]");
  VbRmsConv a{};
  a.T = (int)x.size(0); a.W = (int)x.size(1); a.x = x.data_ptr<float>(); a.nw = nw.data_ptr(); a.eps = (float)eps; a.taps = 1;
  if (y.has_value()) {
    const bool parts = y->dim() == 3;
    TORCH_CHECK(y->is_cuda() && y->size(-1) == a.W && y->size(-2) == a.T && y->stride(-1) == 1, "rms_conv: y");
    if (parts) { CHECK_F32(*y); } else { same(nw, *y, "rms_conv"); }
    a.y = y->data_ptr(); a.y_f32 = parts; a.splits = parts ? (int)y->size(0) : 1; a.split_stride = parts ? y->stride(0) : 0; a.ldy = y->stride(-2);
  }
  if (bias.has_value()) { same(nw, *bias, "rms_conv"); TORCH_CHECK(bias->numel() == a.W && bias->is_contiguous(), "rms_conv: bias [W]"); a.bias = bias->data_ptr(); }
  if (conv.has_value()) {
    same(nw, *conv, "rms_conv");
    TORCH_CHECK(conv->dim() == 2 && conv->size(0) == a.W && conv->size(1) >= 1 && conv->is_contiguous(), "rms_conv: conv [W, taps]");
    a.conv = conv->data_ptr(); a.taps = (int)conv->size(1);
    if (state.has_value() && a.taps > 1) {
      CHECK_F32(*state);
      TORCH_CHECK(state->dim() == 2 && state->stride(1) == 1 && state->size(1) == (int64_t)(a.taps - 1) * a.W, "rms_conv: state [slots, (taps - 1) W]");
      a.state = state->data_ptr<float>(); a.slot_stride = state->stride(0);
    }
    if (cu.has_value()) {
      CHECK_I32(*cu);
      TORCH_CHECK(!y.has_value() && !bias.has_value(), "rms_conv: portions take the stream as it is");
      a.cu = cu->data_ptr<int>(); a.B = (int)cu->numel() - 1;
      if (a.state != nullptr) {
        TORCH_CHECK(slots.has_value() && fresh.has_value() && slots->numel() == a.B && fresh->numel() == a.B, "rms_conv: slots and fresh [B]");
        CHECK_I32(*slots);
        CHECK_I32(*fresh);
        a.slots = slots->data_ptr<int>(); a.fresh = fresh->data_ptr<int>();
      }
    } else {
      TORCH_CHECK(active.has_value() && active->is_cuda() && active->scalar_type() == at::kBool && active->is_contiguous() && active->numel() == a.T, "rms_conv: active [S]");
      TORCH_CHECK(a.taps == 1 || (a.state != nullptr && state->size(0) >= a.T), "rms_conv: steps need a state");
      a.active = reinterpret_cast<const uint8_t*>(active->data_ptr());
    }
  }
  Tensor h = at::empty({a.T, a.W}, nw.options());
  a.h = h.data_ptr();
  verl_count_launches(a.cu != nullptr && a.state != nullptr ? 2 : 1);
  CHECK_RC(vb_rms_conv(dt, &a, cur_stream()), "vb_rms_conv");
  return h;
}

// p [T, r | k | v | za | g | ...], zw [T, H d]
VbDelta delta_args(const Tensor& p, const Tensor& zw, const Tensor& ab, const Tensor& w0, int64_t H, const OptTensor& state, Tensor& out) {
  for (const Tensor* t : {&zw, &ab, &w0}) same(p, *t, "delta");
  const int64_t W = ab.numel(), d = W / H;
  TORCH_CHECK(H > 0 && W == H * d && w0.numel() == W && ab.is_contiguous() && w0.is_contiguous() && p.dim() == 2 && p.stride(1) == 1 && p.size(1) >= 5 * W && zw.dim() == 2 &&
              zw.stride(1) == 1 && zw.size(0) == p.size(0) && zw.size(1) >= W, "delta: rows [r | k | v | a | g]");
  VbDelta a{};
  if (state.has_value()) {
    CHECK_F32(*state);
    TORCH_CHECK(state->dim() == 2 && state->stride(1) == 1 && state->size(1) == W * d, "delta: state [slots, H d d]");
    a.state = state->data_ptr<float>(); a.slot_stride = state->stride(0);
  }
  out = at::empty({p.size(0), W}, p.options());
  a.p = p.data_ptr(); a.ldp = p.stride(0); a.zw = zw.data_ptr(); a.ldz = zw.stride(0); a.ab = ab.data_ptr(); a.w0 = w0.data_ptr(); a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.T = (int)p.size(0); a.H = (int)H; a.d = (int)d;
  return a;
}

Tensor delta_decode(const Tensor& p, const Tensor& zw, const Tensor& ab, const Tensor& w0, int64_t H, const Tensor& norm, double eps, Tensor state, const Tensor& active) {
  const int dt = dtype_of(p);
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor out;
  VbDelta a = delta_args(p, zw, ab, w0, H, state, out);
  same(p, norm, "delta_decode");
  TORCH_CHECK(norm.numel() == ab.numel() && norm.is_contiguous() && active.is_cuda() && active.scalar_type() == at::kBool && active.is_contiguous() && active.numel() == a.T &&
              state.size(0) >= a.T, "delta_decode: active [S]");
  a.active = reinterpret_cast<const uint8_t*>(active.data_ptr()); a.norm = norm.data_ptr(); a.eps = (float)eps;
  verl_count_launches(1);
  CHECK_RC(vb_delta_decode(dt, &a, cur_stream()), "vb_delta_decode");
  return out;
}

Tensor delta_prefill(const Tensor& p, const Tensor& zw, const Tensor& ab, const Tensor& w0, int64_t H, const Tensor& cu, const OptTensor& state, const OptTensor& slots,
                     const OptTensor& fresh) {
  const int dt = dtype_of(p);
  CHECK_I32(cu);
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor out;
  VbDelta a = delta_args(p, zw, ab, w0, H, state, out);
  a.B = (int)cu.numel() - 1;
  a.cu = cu.data_ptr<int>();
  if (slots.has_value()) {
    TORCH_CHECK(state.has_value() && fresh.has_value() && slots->numel() == a.B && fresh->numel() == a.B, "delta_prefill: slots need a state");
    CHECK_I32(*slots);
    CHECK_I32(*fresh);
    a.slots = slots->data_ptr<int>(); a.fresh = fresh->data_ptr<int>();
  }
  if (a.T == 0 || a.B == 0) return out;
  const int nseg = dt == 1 ? vb_delta_chunk_segments(&a) : 0;
  if (nseg > 0) {
    Tensor ws;
    if (nseg > 1) ws = at::empty({(int64_t)a.B * nseg * a.H * 2 * a.d * a.d}, p.options().dtype(at::kFloat));
    const int rc = vb_delta_chunk(&a, nseg, nseg > 1 ? ws.data_ptr<float>() : nullptr, cur_stream());
    if (rc >= 0) {
      verl_count_launches(nseg > 1 ? 3 : 1);
      CHECK_RC(rc, "vb_delta_chunk");
      return out;
    }
  }
  verl_count_launches(1);
  CHECK_RC(vb_delta_scan(dt, &a, cur_stream()), "vb_delta_scan");
  return out;
}

// p [T, q | k | v]; see VbConvPrep. cu given: portions, else one token per slot. Returns (queries [T, H, dim], rows [T or 0, G dim + GV vdim]).
std::tuple<Tensor, Tensor> conv_qkv_prep(const Tensor& p, const OptTensor& conv, double eps, const Tensor& pos, const Tensor& cs, const Tensor& sn, int64_t H, int64_t G,
                                         int64_t GV, int64_t dim, int64_t vdim, bool halves, bool norm, const OptTensor& cu, const OptTensor& state, const OptTensor& slots,
                                         const OptTensor& fresh, const OptTensor& active, const OptTensor& pages, const OptTensor& page_slot, bool want_rows) {
  const int dt = dtype_of(p);
  CHECK_I32(pos);
  CHECK_F32(cs);
  CHECK_F32(sn);
  const int64_t T = p.size(0), C = (H + G) * dim + GV * vdim, width = G * dim + GV * vdim;
  TORCH_CHECK(p.dim() == 2 && p.stride(1) == 1 && p.size(1) >= C && H > 0 && G >= 0 && GV >= 0 && pos.numel() == T && cs.dim() == 2 && cs.is_contiguous() && sn.is_contiguous() &&
              sn.sizes() == cs.sizes() && 2 * cs.size(1) <= dim, "conv_qkv_prep: sizes");
  const c10::cuda::CUDAGuard guard(p.device());
  VbConvPrep a{};
  a.taps = 1;
  if (conv.has_value()) {
    same(p, *conv, "conv_qkv_prep");
    TORCH_CHECK(conv->dim() == 2 && conv->size(0) == C && conv->size(1) >= 1 && conv->is_contiguous(), "conv_qkv_prep: conv [channels, taps]");
    a.conv = conv->data_ptr(); a.taps = (int)conv->size(1);
  }
  if (cu.has_value()) {
    CHECK_I32(*cu);
    a.cu = cu->data_ptr<int>(); a.B = (int)cu->numel() - 1;
  }
  if (state.has_value() && a.taps > 1) {
    CHECK_F32(*state);
    TORCH_CHECK(state->dim() == 2 && state->stride(1) == 1 && state->size(1) == (a.taps - 1) * C, "conv_qkv_prep: state [slots, (taps - 1) channels]");
    a.state = state->data_ptr<float>(); a.slot_stride = state->stride(0);
    if (cu.has_value()) {
      TORCH_CHECK(slots.has_value() && fresh.has_value() && slots->numel() == a.B && fresh->numel() == a.B, "conv_qkv_prep: slots and fresh [B]");
      CHECK_I32(*slots);
      CHECK_I32(*fresh);
      a.slots = slots->data_ptr<int>(); a.fresh = fresh->data_ptr<int>();
    } else {
      TORCH_CHECK(state->size(0) >= T, "conv_qkv_prep: one state row per token of a step");
    }
  }
  if (!cu.has_value()) {
    TORCH_CHECK(active.has_value() && active->is_cuda() && active->scalar_type() == at::kBool && active->is_contiguous() && active->numel() == T, "conv_qkv_prep: active [S]");
    TORCH_CHECK(a.taps == 1 || a.state != nullptr, "conv_qkv_prep: steps need a state");
    a.active = reinterpret_cast<const uint8_t*>(active->data_ptr());
  }
  Tensor q = at::empty({T, H, dim}, p.options()), rows = at::empty({want_rows ? T : 0, width}, p.options());
  a.p = p.data_ptr(); a.ldp = p.stride(0); a.pos = pos.data_ptr<int>(); a.cos_t = cs.data_ptr<float>(); a.sin_t = sn.data_ptr<float>();
  a.half = (int)cs.size(1); a.max_pos = (int)cs.size(0); a.halves = halves;
  a.q = q.data_ptr(); a.ldr = width; a.block_size = 1;
  if (want_rows) a.rows = rows.data_ptr();
  if (pages.has_value()) {
    same(p, *pages, "conv_qkv_prep");
    TORCH_CHECK(pages->dim() == 3 && pages->size(2) == width && pages->stride(2) == 1 && pages->stride(1) == width && page_slot.has_value() && page_slot->is_cuda() &&
                page_slot->scalar_type() == at::kLong && page_slot->is_contiguous() && page_slot->numel() == T, "conv_qkv_prep: pages [blocks, block_size, kv_heads (dim + vdim)]");
    a.pages = pages->data_ptr(); a.page_stride = pages->stride(0); a.block_size = (int)pages->size(1); a.num_slots = pages->size(0) * pages->size(1);
    a.page_slot = lptr(*page_slot);
  }
  a.T = (int)T; a.H = (int)H; a.G = (int)G; a.GV = (int)GV; a.dim = (int)dim; a.vdim = (int)vdim; a.norm = norm; a.eps = (float)eps;
  verl_count_launches(a.cu != nullptr && a.state != nullptr ? 2 : 1);
  CHECK_RC(vb_conv_prep(dt, &a, cur_stream()), "vb_conv_prep");
  return {q, rows};
}

// p [T, q | k | v | ...], decay fp32 [H]
VbLightning lightning_args(const Tensor& p, const Tensor& decay, int64_t d, int64_t e, const OptTensor& state, Tensor& out) {
  CHECK_F32(decay);
  const int64_t H = decay.numel();
  TORCH_CHECK(p.dim() == 2 && p.stride(1) == 1 && d > 0 && e > 0 && p.size(1) >= H * (2 * d + e) && decay.is_contiguous(), "lightning: rows [q | k | v]");
  VbLightning a{};
  if (state.has_value()) {
    CHECK_F32(*state);
    TORCH_CHECK(state->dim() == 2 && state->stride(1) == 1 && state->size(1) == H * d * e, "lightning: state [slots, H d e]");
    a.state = state->data_ptr<float>(); a.slot_stride = state->stride(0);
  }
  out = at::empty({p.size(0), H * e}, p.options());
  a.p = p.data_ptr(); a.ldp = p.stride(0); a.decay = decay.data_ptr<float>(); a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.T = (int)p.size(0); a.H = (int)H; a.d = (int)d; a.e = (int)e;
  return a;
}

Tensor lightning_decode(const Tensor& p, const Tensor& decay, int64_t d, int64_t e, Tensor state, const Tensor& active) {
  const int dt = dtype_of(p);
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor out;
  VbLightning a = lightning_args(p, decay, d, e, state, out);
  TORCH_CHECK(active.is_cuda() && active.scalar_type() == at::kBool && active.is_contiguous() && active.numel() == a.T && state.size(0) >= a.T, "lightning_decode: active [S]");
  a.active = reinterpret_cast<const uint8_t*>(active.data_ptr());
  verl_count_launches(1);
  CHECK_RC(vb_lightning_decode(dt, &a, cur_stream()), "vb_lightning_decode");
  return out;
}

Tensor lightning_prefill(const Tensor& p, const Tensor& decay, int64_t d, int64_t e, const Tensor& cu, const OptTensor& state, const OptTensor& slots, const OptTensor& fresh,
                         bool all_fresh) {
  const int dt = dtype_of(p);
  CHECK_I32(cu);
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor out;
  VbLightning a = lightning_args(p, decay, d, e, state, out);
  a.B = (int)cu.numel() - 1;
  a.cu = cu.data_ptr<int>();
  if (slots.has_value()) {
    TORCH_CHECK(state.has_value() && fresh.has_value() && slots->numel() == a.B && fresh->numel() == a.B, "lightning_prefill: slots need a state");
    CHECK_I32(*slots);
    CHECK_I32(*fresh);
    a.slots = slots->data_ptr<int>(); a.fresh = fresh->data_ptr<int>();
  }
  if (a.T == 0 || a.B == 0) return out;
  if (dt == 1) {
    const int nseg = vb_lightning_chunk_segments(a.T, a.B, a.H, a.d, a.e, all_fresh || !slots.has_value());
    if (nseg > 0) {
      Tensor local;
      if (nseg > 1) local = at::empty({(int64_t)a.B * (nseg - 1) * a.H * d * e}, p.options().dtype(at::kFloat));
      float* ws = nseg > 1 ? local.data_ptr<float>() : nullptr;
      const int rc = d <= 128 ? vb_lightning_tc(&a, nseg, ws, cur_stream()) : vb_lightning_chunk(&a, nseg, ws, cur_stream());
      if (rc >= 0) {
        verl_count_launches(nseg == 1 ? 1 : d <= 128 ? 3 : 2);
        CHECK_RC(rc, "vb_lightning_chunk");
        return out;
      }
    }
  }
  verl_count_launches(1);
  CHECK_RC(vb_lightning_scan(dt, &a, cur_stream()), "vb_lightning_scan");
  return out;
}

struct MlstmShape { int dt; int64_t T, H, d, e; };
MlstmShape mlstm_check(const Tensor& p, const Tensor& gates, const Tensor& ib, const Tensor& fb, const Tensor& norm, int64_t d) {
  MlstmShape s{dtype_of(p), p.size(0), ib.numel(), d, 0};
  s.e = norm.numel() / s.H;
  CHECK_F32(gates);
  same(p, ib, "mlstm");
  same(p, fb, "mlstm");
  same(p, norm, "mlstm");
  TORCH_CHECK(p.dim() == 2 && p.stride(1) == 1 && gates.dim() == 2 && gates.stride(1) == 1 && gates.size(0) == s.T && gates.size(1) >= 2 * s.H && fb.numel() == s.H &&
              norm.numel() == s.H * s.e && p.size(1) >= 2 * s.H * d + 2 * s.H * s.e, "mlstm: [q | k | v | g] rows and [i | f] gates");
  return s;
}
void mlstm_state_check(const Tensor& state, const MlstmShape& s) {
  CHECK_F32(state);
  TORCH_CHECK(state.dim() == 2 && state.stride(1) == 1 && state.size(1) == s.H * (s.d * s.e + s.d + 1), "mlstm: state [slots, H (d e + d + 1)]");
}

Tensor mlstm_decode(const Tensor& p, const Tensor& gates, const Tensor& ib, const Tensor& fb, double cap, Tensor state, const Tensor& active,
                    const Tensor& norm, double eps, int64_t d) {
  const MlstmShape s = mlstm_check(p, gates, ib, fb, norm, d);
  mlstm_state_check(state, s);
  TORCH_CHECK(active.is_cuda() && active.scalar_type() == at::kBool && active.is_contiguous() && active.numel() == s.T && state.size(0) >= s.T, "mlstm_decode: active [S]");
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor out = at::empty({s.T, s.H * s.e}, p.options());
  verl_count_launches(1);
  CHECK_RC(vb_mlstm_decode(s.dt, p.data_ptr(), p.stride(0), gates.data_ptr<float>(), gates.stride(0), ib.data_ptr(), fb.data_ptr(), (float)cap, state.data_ptr<float>(),
                           state.stride(0), reinterpret_cast<const uint8_t*>(active.data_ptr()), norm.data_ptr(), (float)eps, out.data_ptr(), out.stride(0), (int)s.T, (int)s.H,
                           (int)s.d, (int)s.e, cur_stream()), "vb_mlstm_decode");
  return out;
}

// Portion of one or more sequences (cu int32 [B + 1]); slots int32 [B] (or none: nothing is kept), fresh int32 [B]: start from zero.
Tensor mlstm_prefill(const Tensor& p, const Tensor& gates, const Tensor& ib, const Tensor& fb, double cap, const OptTensor& state, const OptTensor& slots,
                     const OptTensor& fresh, const Tensor& cu, const Tensor& norm, double eps, int64_t d, bool all_fresh) {
  const MlstmShape s = mlstm_check(p, gates, ib, fb, norm, d);
  CHECK_I32(cu);
  const int64_t B = cu.numel() - 1;
  if (slots.has_value()) {
    TORCH_CHECK(state.has_value() && fresh.has_value(), "mlstm_prefill: slots need a state");
    mlstm_state_check(*state, s);
    CHECK_I32(*slots);
    CHECK_I32(*fresh);
    TORCH_CHECK(slots->numel() == B && fresh->numel() == B);
  }
  const c10::cuda::CUDAGuard guard(p.device());
  Tensor out = at::empty({s.T, s.H * s.e}, p.options());
  if (s.T == 0 || B == 0) return out;
  const auto f32 = p.options().dtype(at::kFloat);
  float* st = slots.has_value() ? state->data_ptr<float>() : nullptr;
  const int64_t st_stride = slots.has_value() ? state->stride(0) : 0;
  const char* g = reinterpret_cast<const char*>(p.data_ptr()) + (2 * s.H * s.d + s.H * s.e) * p.element_size();
  if (s.dt == 1) {
    const int nseg = vb_mlstm_chunk_segments((int)s.T, (int)B, (int)s.H, (int)s.d, (int)s.e, all_fresh || !slots.has_value());
    if (nseg > 0) {
      Tensor local;
      if (nseg > 1) local = at::empty({B * (nseg - 1) * s.H * (s.d * s.e + s.d + 2)}, f32);
      const int rc = vb_mlstm_chunk(p.data_ptr(), p.stride(0), gates.data_ptr<float>(), gates.stride(0), ib.data_ptr(), fb.data_ptr(), (float)cap, st, st_stride,
                                    iptr(slots), iptr(fresh), cu.data_ptr<int>(), (int)B, nseg, nseg > 1 ? local.data_ptr<float>() : nullptr, norm.data_ptr(), (float)eps,
                                    out.data_ptr(), out.stride(0), (int)s.H, (int)s.d, (int)s.e, cur_stream());
      if (rc >= 0) {
        verl_count_launches(nseg > 1 ? 2 : 1);
        CHECK_RC(rc, "vb_mlstm_chunk");
        return out;
      }
    }
  }
  Tensor o = at::empty({s.T, s.H * s.e}, f32);
  verl_count_launches(slots.has_value() ? 3 : 2);
  CHECK_RC(vb_mlstm_scan(s.dt, p.data_ptr(), p.stride(0), gates.data_ptr<float>(), gates.stride(0), ib.data_ptr(), fb.data_ptr(), (float)cap,
                         st, st_stride, iptr(slots), iptr(fresh), cu.data_ptr<int>(), (int)B,
                         o.data_ptr<float>(), (int)s.T, (int)s.H, (int)s.d, (int)s.e, cur_stream()), "vb_mlstm_scan");
  CHECK_RC(vb_mlstm_out(s.dt, o.data_ptr<float>(), g, p.stride(0), norm.data_ptr(), (float)eps, out.data_ptr(), out.stride(0), (int)s.T, (int)s.H, (int)s.e, cur_stream()),
           "vb_mlstm_out");
  return out;
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(verl_b200, m) {
  m.def("linear_act", &linear_act);
  m.def("linear_split", &linear_split);
  m.def("linear_residual_", &linear_residual_);
  m.def("embed_dyt", &embed_dyt);
  m.def("dynamic_tanh", &dynamic_tanh);
  m.def("rope_pairs_", &rope_pairs_);
  m.def("latent_prep", &latent_prep);
  m.def("gather_pages", &gather_pages);
  m.def("headwise_linear", &headwise_linear);
  m.def("latent_absorb", &latent_absorb);
  m.def("latent_attn_prefill", &latent_attn_prefill);
  m.def("latent_attn_decode", &latent_attn_decode);
  m.def("embed_rms", &embed_rms);
  m.def("linear_partial", &linear_partial);
  m.def("linear_softcap", &linear_softcap);
  m.def("residual_rms_", &residual_rms_);
  m.def("gated_silu", &gated_silu);
  m.def("expert_dispatch", &expert_dispatch);
  m.def("expert_linear", &expert_linear);
  m.def("expert_up", &expert_up);
  m.def("qkv_prep", &qkv_prep);
  m.def("grouped_attn_prefill", &grouped_attn_prefill);
  m.def("grouped_attn_decode", &grouped_attn_decode);
  m.def("linear_bias", &linear_bias);
  m.def("linear_silu", &linear_silu);
  m.def("embed_dyt2", &embed_dyt2);
  m.def("residual_dyt_", &residual_dyt_);
  m.def("gated_rms", &gated_rms);
  m.def("conv_qkv_prep", &conv_qkv_prep);
  m.def("lightning_decode", &lightning_decode);
  m.def("lightning_prefill", &lightning_prefill);
  m.def("mlstm_decode", &mlstm_decode);
  m.def("mlstm_prefill", &mlstm_prefill);
  m.def("linear_tanh", &linear_tanh);
  m.def("whole_norm_prep", &whole_norm_prep);
  m.def("embed_rows", &embed_rows);
  m.def("rms_conv", &rms_conv);
  m.def("delta_prefill", &delta_prefill);
  m.def("delta_decode", &delta_decode);
}
