// Python bindings of the serving library: unpack torch tensors into pointers and pitches, check shapes and bounds that
// the kernels rely on, call the launchers. No math, and no allocation except the one status word per device.
#include <torch/extension.h>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>

#include <atomic>

#include "../attention.h"
#include "../gemm.h"
#include "serve.h"

namespace {

using at::Tensor;
using c10::optional;
using namespace nc::serve;

std::atomic<long long> g_launches{0};

#define NC_CHECK(expr)                                                                                \
  do {                                                                                                \
    ++g_launches;                                                                                     \
    cudaError_t _e = (expr);                                                                          \
    TORCH_CHECK(_e == cudaSuccess, "nanochat_b200 kernel launch failed: ", cudaGetErrorString(_e), " at " #expr); \
  } while (0)

cudaStream_t stream() { return at::cuda::getCurrentCUDAStream().stream(); }

Tensor& status_tensor(const at::Device& dev) {
  static std::vector<Tensor> per_dev(64);
  Tensor& t = per_dev[dev.index()];
  if (!t.defined()) t = torch::zeros({4}, torch::dtype(torch::kInt32).device(dev));
  return t;
}
int* status_ptr(const Tensor& like) { return status_tensor(like.device()).data_ptr<int>(); }

bool is_f32(const Tensor& t) { return t.scalar_type() == at::kFloat; }
// A row matrix the kernels read 8 elements at a time: (rows, n) with dense rows, aligned pitch and base.
void check_rows(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.dim() == 2 && t.stride(1) == 1 && (t.scalar_type() == at::kBFloat16 || is_f32(t)), name,
              ": CUDA bf16 or float rows");
  TORCH_CHECK((t.size(0) == 1 || t.stride(0) % 8 == 0) && t.size(1) % 8 == 0 && (reinterpret_cast<uintptr_t>(t.data_ptr()) & 15) == 0, name,
              ": rows must be multiples of 8 elements and 16-byte aligned");
}
void check_vec(const Tensor& t, int64_t n, const char* name) {
  TORCH_CHECK(t.is_cuda() && is_f32(t) && t.is_contiguous() && t.numel() >= n && (reinterpret_cast<uintptr_t>(t.data_ptr()) & 15) == 0, name,
              ": float vector of at least ", n);
}
long long pitch(const Tensor& t) { return t.size(0) == 1 ? (t.size(1) + 7) / 8 * 8 : t.stride(0); }
void same_type(const Tensor& a, const Tensor& b, const char* name) {
  TORCH_CHECK(a.scalar_type() == b.scalar_type() && a.device() == b.device(), name, ": type or device differs");
}
bool has(const optional<Tensor>& t) { return t.has_value() && t->defined(); }

// pool: (pages, page tokens, width); table: int32 (sequences, max pages); lens: int32 (sequences)
Pages pages_of(const Tensor& pool, const Tensor& table) {
  TORCH_CHECK(pool.is_cuda() && pool.dim() == 3 && pool.is_contiguous() && pool.size(2) % 8 == 0, "pool: dense (pages, tokens, width)");
  TORCH_CHECK(table.is_cuda() && table.scalar_type() == at::kInt && table.dim() == 2 && table.is_contiguous(), "page table: int32 (sequences, pages)");
  const int64_t tokens = pool.size(1);
  TORCH_CHECK(tokens > 0 && (tokens & (tokens - 1)) == 0, "page size must be a power of two");
  int shift = 0;
  while ((int64_t(1) << shift) < tokens) ++shift;
  return Pages{pool.data_ptr(), table.data_ptr<int>(), (int)table.size(1), shift, (int)pool.size(0), (int)pool.size(2)};
}
RowPos positions(const Tensor& lens, const Tensor& table, int64_t per_seq, int64_t rows) {
  TORCH_CHECK(lens.is_cuda() && lens.scalar_type() == at::kInt && lens.is_contiguous() && per_seq > 0 && rows % per_seq == 0 &&
              rows / per_seq <= lens.numel() && rows / per_seq <= table.size(0), "sequence lengths: int32, one per sequence");
  return RowPos{lens.data_ptr<int>(), (int)per_seq};
}
NextWeights next_weights(const optional<Tensor>& t) {
  if (!has(t) || !t->is_contiguous() || (reinterpret_cast<uintptr_t>(t->data_ptr()) & 15)) return {nullptr, 0};
  return {t->data_ptr(), (long long)t->numel() * (long long)t->element_size()};
}

// ------------------------------------------------------------------------------------------------- GEMM, attention
// out (M, N) = A (M, K) B (N, K)^T; grouped: B (groups, N, K), m_group int32, one per 128 rows of A. epi: 0 plain, 1 relu,
// 2 times aux (bf16 like C, may be C itself)
void gemm(const Tensor& A, const Tensor& B, Tensor& C, const optional<Tensor>& m_group, int64_t epi, const optional<Tensor>& aux) {
  check_rows(A, "A"); check_rows(C, "C");
  const bool grouped = has(m_group);
  TORCH_CHECK(A.scalar_type() == at::kBFloat16 && B.scalar_type() == at::kBFloat16 && B.is_cuda() && B.dim() == (grouped ? 3 : 2) &&
              B.stride(-1) == 1 && B.size(-1) == A.size(1) && B.size(-2) == C.size(1) && A.size(0) == C.size(0), "gemm operands");
  const c10::cuda::CUDAGuard guard(A.device());
  nc::GemmDesc d{};
  d.A = A.data_ptr(); d.lda = pitch(A);
  d.B = B.data_ptr(); d.ldb = B.stride(-2);
  d.C = C.data_ptr(); d.ldc = pitch(C); d.c_f32 = is_f32(C);
  d.M = (int)A.size(0); d.N = (int)C.size(1); d.K = (int)A.size(1); d.batch = 1; d.alpha = 1.f;
  if (grouped) {
    TORCH_CHECK(m_group->is_cuda() && m_group->scalar_type() == at::kInt && m_group->is_contiguous() && A.size(0) % 128 == 0 &&
                m_group->numel() * 128 >= A.size(0), "m_group: int32, one per 128 rows");
    d.m_group = m_group->data_ptr<int>(); d.groups = (int)B.size(0); d.bsb = B.stride(0);
  }
  TORCH_CHECK(epi == 0 || (!grouped && !is_f32(C) && (epi == 1 || (epi == 2 && has(aux)))), "gemm epilogue");
  d.epi = epi == 1 ? nc::EPI_RELU : epi == 2 ? nc::EPI_MULAUX : nc::EPI_LINEAR;
  if (has(aux)) {
    check_rows(*aux, "aux"); same_type(*aux, C, "aux");
    TORCH_CHECK(aux->sizes() == C.sizes() && epi == 2, "aux like C");
    d.aux = aux->data_ptr(); d.ldaux = pitch(*aux);
  }
  NC_CHECK(nc::gemm_bf16(d, status_ptr(A), stream()));
}

// q (T, H, D), k and v (S, Hkv, D), o (T, H, D): views with dense innermost dims; softcap 0: none
void attention_capped(const Tensor& q, const Tensor& k, const Tensor& v, Tensor& o, int64_t window_left, double scale, double softcap, double out_scale) {
  for (const Tensor* t : {&q, &k, &v, (const Tensor*)&o}) {
    TORCH_CHECK(t->is_cuda() && t->dim() == 3 && t->scalar_type() == at::kBFloat16 && t->stride(-1) == 1 && (reinterpret_cast<uintptr_t>(t->data_ptr()) & 15) == 0,
                "attention operands: bf16, dense innermost, 16-byte aligned");
    for (int64_t i = 0; i + 1 < t->dim(); ++i) TORCH_CHECK(t->stride(i) % 8 == 0, "attention operands: pitches must be multiples of 8");
  }
  const int64_t T = q.size(0), H = q.size(1), S = k.size(0), Hkv = k.size(1);
  TORCH_CHECK(k.size(2) == q.size(2) && v.size(0) == S && v.size(1) == Hkv && o.size(0) == T && o.size(1) == H && o.size(2) == v.size(2), "attention shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  nc::SplitAttnDesc d{};
  d.a.q = q.data_ptr(); d.a.q_tok = q.stride(0); d.a.q_head = q.stride(1); d.a.q_bat = q.stride(0) * T;
  d.a.k = k.data_ptr(); d.a.k_tok = k.stride(0); d.a.k_head = k.stride(1); d.a.k_bat = k.stride(0) * S;
  d.a.v = v.data_ptr(); d.a.v_tok = v.stride(0); d.a.v_head = v.stride(1); d.a.v_bat = v.stride(0) * S;
  d.a.o = o.data_ptr(); d.a.o_tok = o.stride(0); d.a.o_head = o.stride(1); d.a.o_bat = o.stride(0) * T;
  d.a.B = 1; d.a.Tq = (int)T; d.a.Tk = (int)S; d.a.H = (int)H; d.a.Hkv = (int)Hkv; d.a.D = (int)q.size(2);
  d.Dv = (int)v.size(2);
  d.a.window = (int)window_left; d.a.scale = (float)scale; d.softcap = (float)softcap; d.out_scale = (float)out_scale;
  NC_CHECK(nc::attention_capped_fwd(d, status_ptr(q), stream()));
}

// q (T, H, D), q2 (T, H, D2), k (S, H, D), k2 (S, D2), v (S, H, Dv), o (T, H, Dv): views with dense innermost dims
void attention_split(const Tensor& q, const Tensor& q2, const Tensor& k, const Tensor& k2, const Tensor& v, Tensor& o,
                     int64_t window_left, double scale) {
  for (const Tensor* t : {&q, &q2, &k, &k2, &v, (const Tensor*)&o}) {
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kBFloat16 && t->stride(-1) == 1 && (reinterpret_cast<uintptr_t>(t->data_ptr()) & 15) == 0,
                "attention operands: bf16, dense innermost, 16-byte aligned");
    for (int64_t i = 0; i + 1 < t->dim(); ++i) TORCH_CHECK(t->stride(i) % 8 == 0, "attention operands: pitches must be multiples of 8");
  }
  const int64_t T = q.size(0), H = q.size(1), S = k.size(0);
  TORCH_CHECK(q2.size(0) == T && q2.size(1) == H && k.size(1) == H && k.size(2) == q.size(2) && k2.dim() == 2 && k2.size(0) == S &&
              k2.size(1) == q2.size(2) && v.size(0) == S && v.size(1) == H && o.size(0) == T && o.size(1) == H && o.size(2) == v.size(2),
              "attention shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  nc::SplitAttnDesc d{};
  d.a.q = q.data_ptr(); d.a.q_tok = q.stride(0); d.a.q_head = q.stride(1); d.a.q_bat = q.stride(0) * T;
  d.a.k = k.data_ptr(); d.a.k_tok = k.stride(0); d.a.k_head = k.stride(1); d.a.k_bat = k.stride(0) * S;
  d.a.v = v.data_ptr(); d.a.v_tok = v.stride(0); d.a.v_head = v.stride(1); d.a.v_bat = v.stride(0) * S;
  d.a.o = o.data_ptr(); d.a.o_tok = o.stride(0); d.a.o_head = o.stride(1); d.a.o_bat = o.stride(0) * T;
  d.q2 = q2.data_ptr(); d.q2_tok = q2.stride(0); d.q2_head = q2.stride(1); d.q2_bat = q2.stride(0) * T;
  d.k2 = k2.data_ptr(); d.k2_tok = k2.stride(0); d.k2_bat = k2.stride(0) * S;
  d.a.B = 1; d.a.Tq = (int)T; d.a.Tk = (int)S; d.a.H = (int)H; d.a.Hkv = (int)H; d.a.D = (int)q.size(2);
  d.D2 = (int)q2.size(2); d.Dv = (int)v.size(2);
  d.a.window = (int)window_left; d.a.scale = (float)scale;
  NC_CHECK(nc::attention_split_fwd(d, status_ptr(q), stream()));
}

// ------------------------------------------------------------------------------------------------------------ rows
void embed_norm_(const Tensor& ids, const Tensor& table, int64_t vocab, const Tensor& w, double eps, int64_t n, Tensor& x,
                 const optional<Tensor>& x0, const optional<Tensor>& h) {
  check_rows(table, "table"); check_rows(x, "x");
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous() && ids.numel() == x.size(0), "ids: int64, one per row");
  TORCH_CHECK(is_f32(x) && x.is_contiguous() && x.size(1) <= table.size(1) && n <= x.size(1) && vocab <= table.size(0), "embedding shapes");
  if (has(x0)) TORCH_CHECK(is_f32(*x0) && x0->is_contiguous() && x0->sizes() == x.sizes(), "x0 like x");
  if (has(h)) { same_type(*h, table, "h"); TORCH_CHECK(h->is_contiguous() && h->sizes() == x.sizes(), "h shaped like x"); check_vec(w, x.size(1), "w"); }
  const c10::cuda::CUDAGuard guard(x.device());
  NC_CHECK(embed_norm(is_f32(table), reinterpret_cast<const long long*>(ids.data_ptr<int64_t>()), table.data_ptr(), table.stride(0),
                      (int)vocab, w.data_ptr<float>(), (float)eps, (int)x.size(0), (int)n, (int)x.size(1), x.data_ptr<float>(),
                      has(x0) ? x0->data_ptr<float>() : nullptr, has(h) ? h->data_ptr() : nullptr, stream()));
}

// terms: (gate logits, bias, y) or (gate logits, bias, expert rows, slot, wt)
void gated_residual_norm_(Tensor& x, const std::vector<std::vector<Tensor>>& terms, double mult, const optional<Tensor>& extra,
                          const Tensor& w, double eps, int64_t n, Tensor& h) {
  check_rows(x, "x"); check_rows(h, "h"); check_vec(w, x.size(1), "w");
  TORCH_CHECK(is_f32(x) && x.is_contiguous() && h.is_contiguous() && h.sizes() == x.sizes() && terms.size() <= 2 && n <= x.size(1), "residual shapes");
  if (has(extra)) TORCH_CHECK(is_f32(*extra) && extra->is_contiguous() && extra->sizes() == x.sizes(), "extra like x");
  GatedTerm t[2] = {};
  for (size_t i = 0; i < terms.size(); ++i) {
    const auto& v = terms[i];
    TORCH_CHECK(v.size() == 3 || v.size() == 5, "a term has 3 or 5 tensors");
    check_rows(v[0], "gate"); same_type(v[0], h, "gate"); check_vec(v[1], x.size(1), "bias"); check_rows(v[2], "y"); same_type(v[2], h, "y");
    TORCH_CHECK(v[0].size(0) == x.size(0) && v[0].size(1) == x.size(1) && v[2].size(1) == x.size(1), "term shapes");
    t[i] = {v[0].data_ptr(), pitch(v[0]), v[1].data_ptr<float>(), v[2].data_ptr(), pitch(v[2]), nullptr, nullptr, 0};
    if (v.size() == 5) {
      TORCH_CHECK(v[3].scalar_type() == at::kInt && v[3].is_contiguous() && v[4].sizes() == v[3].sizes() && is_f32(v[4]) && v[4].is_contiguous() &&
                  v[3].dim() == 2 && v[3].size(0) == x.size(0), "slot / wt: (rows, top)");
      t[i].slot = v[3].data_ptr<int>(); t[i].wt = v[4].data_ptr<float>(); t[i].top = (int)v[3].size(1);
    } else {
      TORCH_CHECK(v[2].size(0) == x.size(0), "term rows");
    }
  }
  const c10::cuda::CUDAGuard guard(x.device());
  NC_CHECK(gated_residual_norm(is_f32(h), x.data_ptr<float>(), t, (int)terms.size(), (float)mult,
                               has(extra) ? extra->data_ptr<float>() : nullptr, w.data_ptr<float>(), (float)eps, (int)x.size(0), (int)n,
                               (int)x.size(1), h.data_ptr(), stream()));
}

// x += LN(y) * wy (ids: x = LN(y[ids]) * wy), h = LN(x) * w
void layer_norm_residual_(const optional<Tensor>& ids, const Tensor& y, int64_t vocab, const Tensor& wy, Tensor& x, const Tensor& w, double eps,
                          int64_t n, Tensor& h) {
  check_rows(y, "y"); check_rows(x, "x"); check_rows(h, "h"); check_vec(wy, x.size(1), "wy"); check_vec(w, x.size(1), "w");
  TORCH_CHECK(is_f32(x) && x.is_contiguous() && h.is_contiguous() && h.sizes() == x.sizes() && y.size(1) == x.size(1) && n <= x.size(1) &&
              (is_f32(y) || !is_f32(h)), "layer norm shapes");
  if (has(ids)) {
    TORCH_CHECK(ids->is_cuda() && ids->scalar_type() == at::kLong && ids->is_contiguous() && ids->numel() == x.size(0) && vocab <= y.size(0), "ids: int64, one per row");
  } else {
    TORCH_CHECK(y.size(0) == x.size(0), "y: one row per row of x");
  }
  const c10::cuda::CUDAGuard guard(x.device());
  NC_CHECK(layer_norm_residual(is_f32(h), is_f32(y), has(ids) ? reinterpret_cast<const long long*>(ids->data_ptr<int64_t>()) : nullptr, y.data_ptr(),
                               pitch(y), (int)vocab, wy.data_ptr<float>(), x.data_ptr<float>(), w.data_ptr<float>(), (float)eps, (int)x.size(0), (int)n,
                               (int)x.size(1), h.data_ptr(), stream()));
}

void poly_norm_(const Tensor& z, const Tensor& coef, double eps, int64_t n, Tensor& out) {
  check_rows(z, "z"); check_rows(out, "out");
  TORCH_CHECK(is_f32(z) || !is_f32(out), "poly_norm: float output needs float input");
  TORCH_CHECK(coef.is_cuda() && is_f32(coef) && coef.is_contiguous() && coef.numel() == 4, "poly_norm: four float coefficients");
  TORCH_CHECK(z.sizes() == out.sizes() && n <= z.size(1), "poly_norm shapes");
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(poly_norm(is_f32(out), is_f32(z), z.data_ptr(), pitch(z), coef.data_ptr<float>(), (float)eps, (int)z.size(0), (int)n, (int)z.size(1),
                     out.data_ptr(), pitch(out), stream()));
}

// ---------------------------------------------------------------------------------------------------------- latent
void check_latent(const Tensor& z, int64_t off, int64_t n) { TORCH_CHECK(off >= 0 && off + n <= z.size(1), "latent segments out of range"); }

void latent_post_(const Tensor& z, int64_t q_rank, const optional<Tensor>& q_w, const optional<Tensor>& cq, int64_t c_off, int64_t kv_rank,
                  int64_t kvp, const Tensor& kv_w, double eps, int64_t rot_off, int64_t rot_dim, const Tensor& freq, const Tensor& pool,
                  const Tensor& table, const Tensor& lens, int64_t per_seq, const optional<Tensor>& kv_out) {
  check_rows(z, "z");
  LatentPost d{};
  d.f32 = is_f32(pool); d.z_f32 = is_f32(z);
  d.z = z.data_ptr(); d.ldz = pitch(z); d.rows = (int)z.size(0);
  if (has(cq)) {
    check_rows(*cq, "cq"); same_type(*cq, pool, "cq"); check_vec(*q_w, cq->size(1), "q_w");
    TORCH_CHECK(cq->size(0) == z.size(0) && q_rank <= cq->size(1) && cq->size(1) <= z.size(1), "cq shape");
    d.q_rank = (int)q_rank; d.qp = (int)cq->size(1); d.q_w = q_w->data_ptr<float>(); d.cq = cq->data_ptr(); d.ldcq = pitch(*cq);
  }
  check_latent(z, c_off, kv_rank); check_latent(z, rot_off, rot_dim);
  check_vec(kv_w, kv_rank, "kv_w");
  TORCH_CHECK(is_f32(freq) && freq.is_contiguous() && freq.is_cuda(), "freq");
  d.c_off = (int)c_off; d.kv_rank = (int)kv_rank; d.kvp = (int)kvp; d.kv_w = kv_w.data_ptr<float>(); d.eps = (float)eps;
  d.rot_off = (int)rot_off; d.rot_dim = (int)rot_dim; d.rp = (int)(pool.size(2) - kvp); d.dims = (int)freq.numel() * 2; d.freq = freq.data_ptr<float>();
  d.pg = pages_of(pool, table); d.pos = positions(lens, table, per_seq, z.size(0));
  if (has(kv_out)) {
    check_rows(*kv_out, "kv_out"); same_type(*kv_out, pool, "kv_out");
    TORCH_CHECK(kv_out->size(0) == z.size(0) && kv_out->size(1) == pool.size(2), "kv_out shape");
    d.kv_out = kv_out->data_ptr(); d.ldkv = pitch(*kv_out);
  }
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(latent_post(d, status_ptr(z), stream()));
}

void latent_gather_(const Tensor& pool, const Tensor& table, int64_t seq, int64_t first, Tensor& out) {
  check_rows(out, "out"); same_type(out, pool, "out");
  TORCH_CHECK(seq >= 0 && seq < table.size(0) && out.size(1) == pool.size(2), "gather shape");
  const c10::cuda::CUDAGuard guard(out.device());
  NC_CHECK(latent_gather(is_f32(out), pages_of(pool, table), (int)seq, (int)first, (int)out.size(0), out.data_ptr(), pitch(out),
                         status_ptr(out), stream()));
}

void rotate_heads_(Tensor& q, int64_t heads, int64_t off, const Tensor& freq, const Tensor& table, const Tensor& lens, int64_t per_seq) {
  check_rows(q, "q");
  TORCH_CHECK(q.size(1) % heads == 0 && is_f32(freq) && freq.is_contiguous(), "rotate_heads shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  NC_CHECK(rotate_heads(is_f32(q), q.data_ptr(), pitch(q), (int)q.size(0), (int)heads, (int)(q.size(1) / heads), (int)off,
                        (int)freq.numel() * 2, freq.data_ptr<float>(), positions(lens, table, per_seq, q.size(0)), stream()));
}

void absorb_query_(const Tensor& q, int64_t heads, const Tensor& Wuk, Tensor& qa, bool pdl) {
  check_rows(q, "q"); check_rows(Wuk, "Wuk"); same_type(q, Wuk, "Wuk"); same_type(q, qa, "qa");
  TORCH_CHECK(q.size(1) % heads == 0 && Wuk.is_contiguous() && Wuk.size(0) % heads == 0 && qa.is_contiguous() &&
              qa.numel() == q.size(0) * heads * Wuk.size(1), "absorb_query shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  NC_CHECK(absorb_query(is_f32(q), q.data_ptr(), pitch(q), (int)q.size(0), (int)heads, (int)(q.size(1) / heads), (int)(Wuk.size(0) / heads),
                        Wuk.data_ptr(), (int)Wuk.size(1), qa.data_ptr(), pdl, stream()));
}

void latent_attention_(const Tensor& qa, const Tensor& q, int64_t heads, int64_t dp, int64_t rot_dim, const Tensor& freq, int64_t kvp,
                       const Tensor& pool, const Tensor& table, const Tensor& lens, int64_t per_seq, int64_t window, double scale,
                       int64_t splits, Tensor& ml, Tensor& acc, bool pdl) {
  check_rows(q, "q"); same_type(q, pool, "pool"); same_type(q, qa, "qa");
  const int64_t rows = q.size(0);
  TORCH_CHECK(q.size(1) % heads == 0 && qa.is_contiguous() && qa.numel() == rows * heads * kvp && is_f32(ml) && is_f32(acc) &&
              ml.is_contiguous() && acc.is_contiguous() && splits > 0 && ml.numel() >= rows * heads * splits * 2 &&
              acc.numel() >= rows * heads * splits * kvp && is_f32(freq) && freq.is_contiguous() && pool.size(2) > kvp, "latent_attention shapes");
  LatentAttn d{};
  d.f32 = is_f32(q); d.qa = qa.data_ptr(); d.q = q.data_ptr(); d.ldq = pitch(q); d.head_pitch = (int)(q.size(1) / heads); d.dp = (int)dp;
  d.rot_dim = (int)rot_dim; d.rp = (int)(pool.size(2) - kvp); d.dims = (int)freq.numel() * 2; d.freq = freq.data_ptr<float>();
  d.rows = (int)rows; d.heads = (int)heads; d.kvp = (int)kvp;
  d.pg = pages_of(pool, table); d.pos = positions(lens, table, per_seq, rows);
  d.window = (int)window; d.scale = (float)scale; d.splits = (int)splits; d.ml = ml.data_ptr<float>(); d.acc = acc.data_ptr<float>(); d.pdl = pdl;
  const c10::cuda::CUDAGuard guard(q.device());
  NC_CHECK(latent_attention(d, stream()));
}

void latent_values_(const Tensor& ml, const Tensor& acc, int64_t rows, int64_t heads, int64_t splits, const Tensor& Wuv, Tensor& y, bool pdl,
                    const optional<Tensor>& next) {
  check_rows(Wuv, "Wuv"); check_rows(y, "y"); same_type(Wuv, y, "y");
  const int64_t kvp = Wuv.size(1), vp = Wuv.size(0) / heads;
  TORCH_CHECK(Wuv.is_contiguous() && Wuv.size(0) % heads == 0 && y.size(0) == rows && y.size(1) == heads * vp &&
              ml.numel() >= rows * heads * splits * 2 && acc.numel() >= rows * heads * splits * kvp, "latent_values shapes");
  const c10::cuda::CUDAGuard guard(y.device());
  NC_CHECK(latent_values(is_f32(y), ml.data_ptr<float>(), acc.data_ptr<float>(), (int)rows, (int)heads, (int)splits, (int)kvp,
                         Wuv.data_ptr(), (int)vp, y.data_ptr(), pitch(y), pdl, next_weights(next), stream()));
}

// --------------------------------------------------------------------------------------------------------- experts
void route_topk_(const Tensor& logits, int64_t experts, Tensor& idx, Tensor& wt, const optional<Tensor>& counts, const optional<Tensor>& rank) {
  TORCH_CHECK(logits.is_cuda() && is_f32(logits) && logits.dim() == 2 && logits.stride(1) == 1 && experts <= logits.size(1), "router logits");
  TORCH_CHECK(idx.scalar_type() == at::kInt && idx.is_contiguous() && idx.dim() == 2 && idx.size(0) == logits.size(0) && is_f32(wt) &&
              wt.is_contiguous() && wt.sizes() == idx.sizes(), "idx / wt: (rows, top)");
  if (has(counts)) TORCH_CHECK(counts->scalar_type() == at::kInt && counts->numel() >= experts && has(rank) && rank->sizes() == idx.sizes() &&
                               rank->scalar_type() == at::kInt && rank->is_contiguous(), "counts / rank");
  const c10::cuda::CUDAGuard guard(logits.device());
  NC_CHECK(route_topk(logits.data_ptr<float>(), logits.size(0) == 1 ? logits.size(1) : logits.stride(0), (int)logits.size(0), (int)experts,
                      (int)idx.size(1), idx.data_ptr<int>(), wt.data_ptr<float>(), has(counts) ? counts->data_ptr<int>() : nullptr,
                      has(rank) ? rank->data_ptr<int>() : nullptr, stream()));
}

void group_rows(const Tensor& h, const Tensor& idx, const Tensor& rank, const Tensor& counts, Tensor& offsets, Tensor& tile_group,
                Tensor& slot, Tensor& xg) {
  check_rows(h, "h"); check_rows(xg, "xg");
  const int64_t rows = h.size(0), top = idx.size(1), experts = counts.numel();
  for (const Tensor* t : {&idx, &rank, &counts, (const Tensor*)&offsets, (const Tensor*)&tile_group, (const Tensor*)&slot})
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kInt && t->is_contiguous(), "group_rows: int32 indices");
  TORCH_CHECK(h.scalar_type() == at::kBFloat16 && xg.scalar_type() == at::kBFloat16 && xg.is_contiguous() && xg.size(1) == h.size(1) &&
              xg.size(0) == tile_group.numel() * 128 && xg.size(0) >= rows * top + experts * 127 && offsets.numel() >= experts &&
              slot.numel() == rows * top && rank.numel() == rows * top && idx.size(0) == rows, "group_rows shapes");
  const c10::cuda::CUDAGuard guard(h.device());
  NC_CHECK(plan_groups(counts.data_ptr<int>(), (int)experts, offsets.data_ptr<int>(), tile_group.data_ptr<int>(), (int)tile_group.numel(), stream()));
  NC_CHECK(gather_groups(h.data_ptr(), pitch(h), (int)rows, (int)top, (int)h.size(1), idx.data_ptr<int>(), rank.data_ptr<int>(),
                         offsets.data_ptr<int>(), slot.data_ptr<int>(), xg.data_ptr(), stream()));
}

void silu_mul_(const Tensor& gu, const Tensor& tile_group, Tensor& act) {
  check_rows(gu, "gu"); check_rows(act, "act");
  TORCH_CHECK(gu.scalar_type() == at::kBFloat16 && act.scalar_type() == at::kBFloat16 && gu.is_contiguous() && act.is_contiguous() &&
              gu.size(0) == act.size(0) && gu.size(1) == 2 * act.size(1) && tile_group.scalar_type() == at::kInt &&
              tile_group.numel() * 128 >= gu.size(0), "silu_mul shapes");
  const c10::cuda::CUDAGuard guard(gu.device());
  NC_CHECK(silu_mul(gu.data_ptr(), (int)gu.size(0), (int)act.size(1), tile_group.data_ptr<int>(), act.data_ptr(), stream()));
}

Routing routing_of(const Tensor& idx, const Tensor& wt, int64_t rows, int64_t experts) {
  TORCH_CHECK(idx.scalar_type() == at::kInt && idx.is_contiguous() && idx.dim() == 2 && idx.size(0) == rows && is_f32(wt) && wt.is_contiguous() &&
              wt.sizes() == idx.sizes(), "routing: (rows, top)");
  return Routing{idx.data_ptr<int>(), wt.data_ptr<float>(), (int)experts, (int)idx.size(1)};
}

void expert_gate_up_(const Tensor& h, const Tensor& Wgu, const Tensor& idx, const Tensor& wt, Tensor& act) {
  check_rows(h, "h"); check_rows(act, "act"); same_type(h, Wgu, "Wgu"); same_type(h, act, "act");
  TORCH_CHECK(Wgu.dim() == 3 && Wgu.is_contiguous() && Wgu.size(2) == h.size(1) && Wgu.size(1) == 2 * act.size(1) && act.is_contiguous() &&
              act.size(0) == idx.numel(), "expert_gate_up shapes");
  const c10::cuda::CUDAGuard guard(h.device());
  NC_CHECK(expert_gate_up(is_f32(h), h.data_ptr(), pitch(h), (int)h.size(0), (int)h.size(1), Wgu.data_ptr(), (int)act.size(1),
                          routing_of(idx, wt, h.size(0), Wgu.size(0)), act.data_ptr(), stream()));
}

void expert_down_(const Tensor& act, const Tensor& Wdown, const Tensor& idx, const Tensor& wt, Tensor& y) {
  check_rows(act, "act"); same_type(act, Wdown, "Wdown"); check_rows(y, "y"); same_type(y, act, "y");
  TORCH_CHECK(act.is_contiguous() && act.size(0) == idx.numel() && Wdown.dim() == 3 && Wdown.is_contiguous() && Wdown.size(2) == act.size(1) &&
              y.size(1) == Wdown.size(1), "expert_down shapes");
  ExpertDown d{};
  d.f32 = is_f32(act); d.act = act.data_ptr(); d.rows = (int)y.size(0); d.fp = (int)act.size(1); d.Wdown = Wdown.data_ptr(); d.N = (int)Wdown.size(1);
  d.rt = routing_of(idx, wt, y.size(0), Wdown.size(0));
  d.y = y.data_ptr(); d.ldy = pitch(y);
  const c10::cuda::CUDAGuard guard(y.device());
  NC_CHECK(expert_down(d, stream()));
}
void check_gate(const Tensor& x, const Tensor& g, const Tensor& bias, const optional<Tensor>& extra, int64_t rows, int64_t n) {
  TORCH_CHECK(is_f32(x) && x.is_cuda() && x.is_contiguous() && x.dim() == 2 && x.size(0) == rows && x.size(1) == n, "residual: float (rows, n)");
  TORCH_CHECK(is_f32(g) && g.dim() == 2 && g.stride(1) == 1 && g.size(0) == rows && g.size(1) == n && is_f32(bias) && bias.is_contiguous() &&
              bias.numel() >= n, "gate logits / bias: float");
  if (has(extra)) TORCH_CHECK(is_f32(*extra) && extra->is_contiguous() && extra->sizes() == x.sizes(), "extra like the residual");
}
// out[b] = mult * sigmoid(g + bias) * (the row's weighted experts on h) (+ extra), float (rows, n), rows <= 8
void expert_rows_(const Tensor& h, const Tensor& Wgu, const Tensor& Wdown, const Tensor& idx, const Tensor& wt, Tensor& act, Tensor& out,
                  const Tensor& g, const Tensor& bias, double mult, const optional<Tensor>& extra) {
  check_rows(h, "h"); check_rows(act, "act");
  for (const Tensor* t : {&h, &Wgu, &Wdown, (const Tensor*)&act}) TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kBFloat16, "expert_rows: bf16");
  TORCH_CHECK(Wgu.dim() == 3 && Wgu.is_contiguous() && Wgu.size(2) == h.size(1) && Wgu.size(1) == 2 * act.size(1) && Wdown.dim() == 3 && Wdown.is_contiguous() &&
              Wdown.size(0) == Wgu.size(0) && Wdown.size(2) == act.size(1) && act.is_contiguous() && act.size(0) == idx.numel(), "expert_rows shapes");
  check_gate(out, g, bias, extra, h.size(0), Wdown.size(1));
  const Routing rt = routing_of(idx, wt, h.size(0), Wgu.size(0));
  ExpertRows d{};
  d.h = h.data_ptr(); d.ldh = pitch(h); d.rows = (int)h.size(0); d.top = rt.top; d.experts = rt.experts; d.K = (int)h.size(1); d.fp = (int)act.size(1);
  d.N = (int)Wdown.size(1); d.Wgu = Wgu.data_ptr(); d.Wdown = Wdown.data_ptr(); d.idx = rt.idx; d.wt = rt.wt; d.act = act.data_ptr();
  d.out = out.data_ptr<float>(); d.ldo = out.stride(0); d.g = g.data_ptr<float>(); d.ldg = g.stride(0); d.bias = bias.data_ptr<float>(); d.mult = (float)mult;
  d.extra = has(extra) ? extra->data_ptr<float>() : nullptr;
  const c10::cuda::CUDAGuard guard(h.device());
  ++g_launches;
  NC_CHECK(expert_rows(d, stream()));
}

// ------------------------------------------------------------------------------------------------------------ gemv
GemvDesc gemv_of(const Tensor& x, const Tensor& W, const optional<Tensor>& next, bool any_rows = false) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 2 && x.stride(1) == 1 && W.is_cuda() && W.scalar_type() == at::kBFloat16, "gemv operands");
  check_rows(x, "x"); check_rows(W, "W");
  TORCH_CHECK(x.size(1) == W.size(1) && (any_rows || x.size(0) <= 8), "gemv shapes");
  GemvDesc d{};
  d.x = x.data_ptr(); d.ldx = pitch(x); d.W = W.data_ptr(); d.ldw = pitch(W); d.rows = (int)x.size(0); d.N = (int)W.size(0); d.K = (int)x.size(1);
  d.next = next_weights(next); d.pdl = true; d.accumulate = true;
  return d;
}
int store_kind(GemvDesc& d, Tensor& out) {
  TORCH_CHECK(out.is_cuda() && out.dim() == 2 && out.stride(1) == 1 && out.size(0) == d.rows && out.size(1) == d.N &&
              (is_f32(out) || out.scalar_type() == at::kBFloat16), "gemv output");
  d.out = out.data_ptr(); d.ldo = out.stride(0);
  return is_f32(out) ? GEMV_STORE_F32 : GEMV_STORE_BF16;
}
// out = (x / rms(x) * w) W^T; h: the normed rows as bf16.
void gemv_norm(const Tensor& x, const Tensor& w, double eps, int64_t n, const Tensor& W, Tensor& out, const optional<Tensor>& h,
               const optional<Tensor>& next) {
  GemvDesc d = gemv_of(x, W, next);
  TORCH_CHECK(is_f32(x), "gemv_norm: float rows"); check_vec(w, x.size(1), "w");
  d.w = w.data_ptr<float>(); d.eps = (float)eps; d.n_real = (int)n;
  if (has(h)) {
    TORCH_CHECK(h->scalar_type() == at::kBFloat16 && h->is_contiguous() && h->sizes() == x.sizes(), "h: bf16 like x");
    d.h_out = h->data_ptr(); d.ldh = x.size(1);
  }
  const int epi = store_kind(d, out);
  const c10::cuda::CUDAGuard guard(x.device());
  NC_CHECK(gemv(d, PRE_NORM, epi, stream()));
}
// The query half of a latent layer's decode step: q = (norm of z[:, :q_rank]) Wq^T, and the step's store entries.
void gemv_query_store(const Tensor& z, int64_t q_rank, const Tensor& q_w, double eps, const Tensor& Wq, Tensor& q, int64_t c_off, int64_t kv_rank,
                      int64_t kvp, const Tensor& kv_w, int64_t rot_off, int64_t rot_dim, const Tensor& freq, const Tensor& pool,
                      const Tensor& table, const Tensor& lens, const optional<Tensor>& next) {
  TORCH_CHECK(is_f32(z) && z.dim() == 2 && z.stride(1) == 1 && Wq.size(1) <= z.size(1), "z: float rows");
  const Tensor x = z.narrow(1, 0, Wq.size(1));
  GemvDesc d = gemv_of(x, Wq, next);
  d.ldx = z.size(0) == 1 ? d.ldx : z.stride(0);
  check_vec(q_w, Wq.size(1), "q_w"); check_vec(kv_w, kv_rank, "kv_w");
  d.w = q_w.data_ptr<float>(); d.eps = (float)eps; d.n_real = (int)q_rank;
  check_latent(z, c_off, kv_rank); check_latent(z, rot_off, rot_dim);
  TORCH_CHECK(pool.scalar_type() == at::kBFloat16 && pool.size(2) > kvp && kv_rank <= kvp && is_f32(freq) && freq.is_contiguous() && freq.numel() * 2 <= rot_dim &&
              rot_dim <= pool.size(2) - kvp && rot_off >= c_off, "store shapes");
  LatentStore s{};
  s.z = z.data_ptr<float>() + c_off; s.ldz = z.stride(0); s.kv_rank = (int)kv_rank; s.kvp = (int)kvp; s.kv_w = kv_w.data_ptr<float>(); s.eps = (float)eps;
  s.rot_off = (int)(rot_off - c_off); s.rot_dim = (int)rot_dim; s.rp = (int)(pool.size(2) - kvp); s.dims = (int)freq.numel() * 2; s.freq = freq.data_ptr<float>();
  s.pg = pages_of(pool, table); s.pos = positions(lens, table, 1, z.size(0)); s.status = status_ptr(z);
  d.store = &s;
  const int epi = store_kind(d, q);
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(gemv(d, PRE_NORM, epi, stream()));
}
// x[b] (+)= mult * sigmoid(g + bias) * (y W^T) (+ extra); y: bf16 rows. pdl: false where the kernel before is not the only
// one this waits for
void gemv_residual(const Tensor& y, const Tensor& W, Tensor& x, const Tensor& g, const Tensor& bias, double mult, const optional<Tensor>& extra,
                   const optional<Tensor>& next, bool accumulate, bool pdl) {
  GemvDesc d = gemv_of(y, W, next);
  TORCH_CHECK(y.scalar_type() == at::kBFloat16, "y: bf16 rows");
  check_gate(x, g, bias, extra, y.size(0), W.size(0));
  d.resid = x.data_ptr<float>(); d.ldr = x.stride(0); d.g = g.data_ptr<float>(); d.ldg = g.stride(0); d.bias = bias.data_ptr<float>();
  d.mult = (float)mult; d.extra = has(extra) ? extra->data_ptr<float>() : nullptr; d.accumulate = accumulate; d.pdl = pdl;
  const c10::cuda::CUDAGuard guard(x.device());
  NC_CHECK(gemv(d, PRE_PLAIN, GEMV_RESIDUAL, stream()));
}

// out = x W^T, x bf16 rows
void gemv_plain(const Tensor& x, const Tensor& W, Tensor& out, const optional<Tensor>& next) {
  GemvDesc d = gemv_of(x, W, next, true);
  TORCH_CHECK(x.scalar_type() == at::kBFloat16, "x: bf16 rows");
  const int epi = store_kind(d, out);
  const c10::cuda::CUDAGuard guard(x.device());
  NC_CHECK(gemv(d, PRE_PLAIN, epi, stream()));
}
// out = relu(x Wg^T) * (x Wu^T), W = [Wg; Wu]
void gemv_relu_glu_(const Tensor& x, const Tensor& W, Tensor& out, const optional<Tensor>& next) {
  GemvDesc d = gemv_of(x, W, next);
  TORCH_CHECK(x.scalar_type() == at::kBFloat16 && W.size(0) % 2 == 0, "x: bf16 rows; W: gate rows, then up rows");
  d.N = (int)(W.size(0) / 2);
  TORCH_CHECK(store_kind(d, out) == GEMV_STORE_BF16, "out: bf16");
  const c10::cuda::CUDAGuard guard(x.device());
  NC_CHECK(gemv_relu_glu(d, stream()));
}

// ------------------------------------------------------------------------------------------------ recurrences, windows
// A module's sizes travel as one list: delta [heads, kv_heads, dim, dp, vdim, vp, taps, a_off].
StateRef state_ref(const Tensor& t, int64_t seqs, int64_t per_seq, const char* name) {
  TORCH_CHECK(t.is_cuda() && is_f32(t) && t.dim() >= 2 && t.size(0) >= seqs && t.stride(0) % 4 == 0 && (reinterpret_cast<uintptr_t>(t.data_ptr()) & 15) == 0, name,
              ": float, one row per sequence, 16-byte aligned");
  int64_t n = 1;
  for (int64_t i = t.dim() - 1; i >= 1; --i) {
    TORCH_CHECK(t.stride(i) == n, name, ": dense per sequence");
    n *= t.size(i);
  }
  TORCH_CHECK(n == per_seq && (seqs == 1 || t.stride(0) >= n), name, ": size");
  return StateRef{t.data_ptr<float>(), (long long)t.stride(0)};
}
RowPos row_pos(const Tensor& lens, int64_t per_seq, int64_t rows) {
  TORCH_CHECK(lens.is_cuda() && lens.scalar_type() == at::kInt && lens.is_contiguous() && per_seq > 0 && rows % per_seq == 0 && rows / per_seq <= lens.numel(),
              "sequence lengths: int32, one per sequence");
  return RowPos{lens.data_ptr<int>(), (int)per_seq};
}
DeltaInputs delta_inputs(const Tensor& z, const std::vector<int64_t>& size, const Tensor& conv, const optional<Tensor>& ba, const Tensor& neg_a,
                         const Tensor& dt_bias, const Tensor& ring, const Tensor& lens, int64_t per_seq, bool f32) {
  check_rows(z, "z");
  TORCH_CHECK(size.size() == 8, "delta rule: eight sizes");
  DeltaInputs d{};
  d.f32 = f32; d.z_f32 = is_f32(z); d.z = z.data_ptr(); d.ldz = pitch(z); d.rows = (int)z.size(0);
  d.heads = (int)size[0]; d.kv_heads = (int)size[1]; d.dim = (int)size[2]; d.dp = (int)size[3]; d.vdim = (int)size[4]; d.vp = (int)size[5]; d.taps = (int)size[6];
  d.a_off = (int)size[7];
  const int64_t channels = 2 * size[1] * size[3] + size[0] * size[5];
  TORCH_CHECK(size[0] > 0 && size[1] > 0 && size[6] > 0 && channels <= z.size(1), "delta rule: sizes");
  check_vec(conv, size[6] * channels, "conv"); check_vec(neg_a, size[0], "neg_a"); check_vec(dt_bias, size[0], "dt_bias");
  d.conv = conv.data_ptr<float>(); d.neg_a = neg_a.data_ptr<float>(); d.dt_bias = dt_bias.data_ptr<float>();
  if (has(ba)) {
    TORCH_CHECK(ba->is_cuda() && is_f32(*ba) && ba->dim() == 2 && ba->stride(1) == 1 && ba->size(0) == z.size(0) && size[7] + size[0] <= ba->size(1), "ba: float rows");
    d.ba = ba->data_ptr<float>(); d.ldba = ba->size(0) == 1 ? ba->size(1) : ba->stride(0);
  }
  d.pos = row_pos(lens, per_seq, z.size(0));
  d.ring = state_ref(ring, z.size(0) / per_seq, size[6] * channels, "ring");
  return d;
}
// Where prepared inputs go: rows x channels in the compute type, or (uint8) tiles.
bool check_prepared(const Tensor& out, int64_t rows, int64_t per_seq, int64_t H, int64_t G, int64_t dp, int64_t vp, bool f32) {
  TORCH_CHECK(out.is_cuda() && out.is_contiguous() && (reinterpret_cast<uintptr_t>(out.data_ptr()) & 15) == 0, "prepared inputs: dense, 16-byte aligned");
  if (out.scalar_type() == at::kByte) {
    TORCH_CHECK(!f32 && recurrence_chunks_supported((int)dp) && (size_t)out.numel() >= recurrence_tiles((int)(rows / per_seq), (int)per_seq, (int)H, (int)G, (int)dp, (int)vp),
                "tiles: too small, or sizes the chunk kernels do not take");
    return true;
  }
  TORCH_CHECK(is_f32(out) == f32 && (f32 || out.scalar_type() == at::kBFloat16) && out.dim() == 2 && out.size(0) == rows && out.size(1) == 2 * G * dp + H * vp,
              "prepared inputs: rows x channels");
  return false;
}
void delta_prepare_(const Tensor& z, const std::vector<int64_t>& size, const Tensor& conv, const Tensor& ba, const Tensor& neg_a, const Tensor& dt_bias,
                    const Tensor& ring, const Tensor& lens, int64_t per_seq, Tensor& out, Tensor& norms, Tensor& beta_g) {
  const DeltaInputs d = delta_inputs(z, size, conv, ba, neg_a, dt_bias, ring, lens, per_seq, is_f32(out));
  const bool tiles = check_prepared(out, z.size(0), per_seq, size[0], size[1], size[3], size[5], is_f32(out));
  TORCH_CHECK(is_f32(norms) && norms.is_contiguous() && norms.numel() >= z.size(0) * 2 * size[1] && is_f32(beta_g) && beta_g.is_contiguous() &&
              beta_g.numel() >= z.size(0) * 2 * size[0], "delta rule: outputs");
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(delta_prepare(d, tiles, out.data_ptr(), norms.data_ptr<float>(), beta_g.data_ptr<float>(), stream()));
}
// z: q, k (heads x dp each), v (heads x vp) side by side
void decay_prepare_(const Tensor& z, int64_t heads, int64_t dp, int64_t vp, int64_t per_seq, Tensor& out) {
  check_rows(z, "z");
  TORCH_CHECK(heads > 0 && z.size(1) == heads * (2 * dp + vp) && per_seq > 0 && z.size(0) % per_seq == 0, "decay_prepare shapes");
  const bool tiles = check_prepared(out, z.size(0), per_seq, heads, heads, dp, vp, is_f32(z));
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(decay_prepare(is_f32(z), z.data_ptr(), pitch(z), (int)z.size(0), (int)per_seq, (int)heads, (int)dp, (int)vp, tiles, out.data_ptr(), stream()));
}
// size: [heads, kv_heads, dp, vp]; act: what a prepare kernel left; norms and beta_g, or log_decay. Tiles need scratch.
void recurrence_(const Tensor& act, const std::vector<int64_t>& size, const optional<Tensor>& norms, const optional<Tensor>& beta_g,
                 const optional<Tensor>& log_decay, const Tensor& state, const Tensor& lens, int64_t per_seq, Tensor& o, const optional<Tensor>& scratch) {
  check_rows(o, "o");
  TORCH_CHECK(size.size() == 4 && size[0] > 0 && size[1] > 0, "recurrence: four sizes");
  const int64_t H = size[0], G = size[1], dp = size[2], vp = size[3], rows = o.size(0);
  TORCH_CHECK(o.size(1) == H * vp, "recurrence shapes");
  Recurrence d{};
  d.f32 = is_f32(o); d.act = act.data_ptr(); d.lda = 2 * G * dp + H * vp; d.q_off = 0; d.k_off = (int)(G * dp); d.v_off = (int)(2 * G * dp);
  d.rows = (int)rows; d.heads = (int)H; d.kv_heads = (int)G; d.dp = (int)dp; d.vp = (int)vp;
  d.pos = row_pos(lens, per_seq, rows);
  const bool tiles = check_prepared(act, rows, per_seq, H, G, dp, vp, d.f32);
  const bool delta = has(beta_g);
  if (delta) {
    TORCH_CHECK(has(norms), "delta rule: norms");
    check_vec(*norms, rows * 2 * G, "norms"); check_vec(*beta_g, rows * 2 * H, "beta_g");
    d.norms = norms->data_ptr<float>(); d.beta_g = beta_g->data_ptr<float>();
  } else {
    TORCH_CHECK(has(log_decay), "fixed decay: log_decay");
    check_vec(*log_decay, H, "log_decay");
    d.log_decay = log_decay->data_ptr<float>();
  }
  d.state = state_ref(state, rows / per_seq, H * dp * vp, "state");
  d.o = o.data_ptr(); d.ldo = pitch(o);
  const c10::cuda::CUDAGuard guard(o.device());
  if (tiles) {
    TORCH_CHECK(has(scratch) && scratch->is_cuda() && scratch->is_contiguous() && (reinterpret_cast<uintptr_t>(scratch->data_ptr()) & 15) == 0 &&
                (size_t)(scratch->numel() * scratch->element_size()) >= recurrence_scratch((int)(rows / per_seq), (int)per_seq, (int)H, delta), "scratch: too small");
    ++g_launches;
    NC_CHECK(recurrence_chunks(d, scratch->data_ptr(), status_ptr(o), stream()));
  } else {
    NC_CHECK(recurrence_scan(d, stream()));
  }
}
// y = o / rms(o) * w * act(gate) * out_scale in `groups` groups of n real entries
void norm_gate_(const Tensor& o, const Tensor& gate, const Tensor& w, double eps, int64_t groups, int64_t n, bool sigmoid, double out_scale, Tensor& y) {
  check_rows(o, "o"); check_rows(gate, "gate"); check_rows(y, "y"); same_type(o, gate, "gate"); same_type(o, y, "y");
  TORCH_CHECK(groups > 0 && o.size(1) % groups == 0 && gate.sizes() == o.sizes() && y.sizes() == o.sizes(), "norm_gate shapes");
  check_vec(w, o.size(1) / groups, "w");
  const c10::cuda::CUDAGuard guard(o.device());
  NC_CHECK(norm_gate(is_f32(o), o.data_ptr(), pitch(o), gate.data_ptr(), pitch(gate), w.data_ptr<float>(), (float)eps, (int)o.size(0), (int)groups, (int)n,
                     (int)(o.size(1) / groups), sigmoid ? 1 : 0, (float)out_scale, y.data_ptr(), pitch(y), nullptr, stream()));
}
// The same for the delta rule's heads (silu), and the ring keeps the rows' last convolution inputs (z's channels).
void delta_finish(const Tensor& o, const Tensor& gate, const Tensor& w, double eps, Tensor& y, const Tensor& z, const std::vector<int64_t>& size,
                  const Tensor& conv, const Tensor& neg_a, const Tensor& dt_bias, const Tensor& ring, const Tensor& lens, int64_t per_seq) {
  check_rows(o, "o"); check_rows(gate, "gate"); check_rows(y, "y"); same_type(o, gate, "gate"); same_type(o, y, "y"); same_type(o, z, "z");
  const DeltaInputs d = delta_inputs(z, size, conv, c10::nullopt, neg_a, dt_bias, ring, lens, per_seq, is_f32(o));
  TORCH_CHECK(o.size(0) == z.size(0) && o.size(1) == size[0] * size[5] && gate.sizes() == o.sizes() && y.sizes() == o.sizes(), "delta_finish shapes");
  check_vec(w, size[5], "w");
  const c10::cuda::CUDAGuard guard(o.device());
  NC_CHECK(norm_gate(is_f32(o), o.data_ptr(), pitch(o), gate.data_ptr(), pitch(gate), w.data_ptr<float>(), (float)eps, (int)o.size(0), (int)size[0], (int)size[4],
                     (int)size[5], 0, 1.f, y.data_ptr(), pitch(y), &d, stream()));
}
// One token per row, z to y.
void delta_step_(const Tensor& z, const std::vector<int64_t>& size, const Tensor& conv, const Tensor& ba, const Tensor& neg_a, const Tensor& dt_bias,
                 const Tensor& ring, const Tensor& state, const Tensor& lens, const Tensor& norm, double eps, int64_t gate_off, Tensor& y) {
  check_rows(y, "y");
  DeltaStep d{};
  d.in = delta_inputs(z, size, conv, ba, neg_a, dt_bias, ring, lens, 1, is_f32(y));
  d.state = state_ref(state, z.size(0), size[0] * size[3] * size[5], "state");
  check_vec(norm, size[5], "norm");
  TORCH_CHECK(gate_off >= 0 && gate_off + size[0] * size[5] <= z.size(1) && y.size(0) == z.size(0) && y.size(1) == size[0] * size[5], "delta_step shapes");
  d.norm = norm.data_ptr<float>(); d.eps = (float)eps; d.gate_off = (int)gate_off; d.y = y.data_ptr(); d.ldy = pitch(y);
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(delta_step(d, stream()));
}

// size: [heads, kv_heads, dp, q_off, k_off, window]; real: [scale, softcap, out_scale]
WindowAttn window_of(const Tensor& z, const std::vector<int64_t>& size, const std::vector<double>& real, const Tensor& freq, const Tensor& pool,
                     const Tensor& table, const Tensor& lens, int64_t per_seq) {
  check_rows(z, "z");
  TORCH_CHECK(size.size() == 6 && real.size() == 3 && size[0] > 0 && size[1] > 0 && is_f32(freq) && freq.is_cuda() && freq.is_contiguous() &&
              freq.numel() % 2 == 0, "window attention: sizes");
  TORCH_CHECK(size[3] >= 0 && size[3] + size[0] * size[2] <= z.size(1) && size[4] >= 0 && size[4] + size[1] * size[2] <= z.size(1), "window attention: segments of z");
  WindowAttn d{};
  d.f32 = is_f32(pool); d.z_f32 = is_f32(z); d.z = z.data_ptr(); d.ldz = pitch(z); d.q_off = (int)size[3]; d.k_off = (int)size[4];
  d.rows = (int)z.size(0); d.heads = (int)size[0]; d.kv_heads = (int)size[1]; d.dp = (int)size[2]; d.dims = (int)freq.numel(); d.freq = freq.data_ptr<float>();
  d.pg = pages_of(pool, table); d.pos = positions(lens, table, per_seq, z.size(0)); d.window = (int)size[5];
  d.scale = (float)real[0]; d.softcap = (float)real[1]; d.out_scale = (float)real[2];
  return d;
}
void window_out(WindowAttn& d, Tensor& y, const Tensor& pool) {
  check_rows(y, "y"); same_type(y, pool, "y");
  TORCH_CHECK(y.size(0) == d.rows && y.size(1) == (int64_t)d.heads * d.dp, "window attention: output");
  d.y = y.data_ptr(); d.ldy = pitch(y);
}
void window_post_(Tensor& z, const std::vector<int64_t>& size, const std::vector<double>& real, const Tensor& freq, const Tensor& pool, const Tensor& table,
                  const Tensor& lens, int64_t per_seq, const optional<Tensor>& dense) {
  const WindowAttn d = window_of(z, size, real, freq, pool, table, lens, per_seq);
  same_type(z, pool, "pool");
  if (has(dense)) {
    check_rows(*dense, "dense"); same_type(*dense, pool, "dense");
    TORCH_CHECK(dense->size(0) == z.size(0) && dense->size(1) == pool.size(2), "dense: one entry per row");
  }
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(window_post(d, has(dense) ? dense->data_ptr() : nullptr, has(dense) ? pitch(*dense) : 0, status_ptr(z), stream()));
}
void window_attention_(const Tensor& z, const std::vector<int64_t>& size, const std::vector<double>& real, const Tensor& freq, const Tensor& pool,
                       const Tensor& table, const Tensor& lens, int64_t per_seq, Tensor& y) {
  WindowAttn d = window_of(z, size, real, freq, pool, table, lens, per_seq);
  same_type(z, pool, "pool");
  window_out(d, y, pool);
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(window_attention(d, stream()));
}
// size: [heads, dp, vdim, vp, q_off, k_off, v_off, gate_off]; real: [eps, out_scale]
DecayStep decay_of(const Tensor& z, const std::vector<int64_t>& size, const std::vector<double>& real, const Tensor& log_decay, const Tensor& state,
                   const Tensor& lens, const Tensor& norm, Tensor& o, Tensor& done, Tensor& y) {
  check_rows(z, "z"); check_rows(y, "y");
  TORCH_CHECK(size.size() == 8 && real.size() == 2 && size[0] > 0, "fixed decay: sizes");
  const int64_t H = size[0], dp = size[1], vp = size[3], width = H * vp, rows = z.size(0);
  for (int i = 4; i < 8; ++i) TORCH_CHECK(size[i] >= 0 && size[i] + H * (i < 6 ? dp : vp) <= z.size(1), "fixed decay: segments of z");
  check_vec(log_decay, H, "log_decay"); check_vec(norm, width, "norm"); check_vec(o, rows * width, "o");
  TORCH_CHECK(done.is_cuda() && done.scalar_type() == at::kInt && done.is_contiguous() && done.numel() >= rows && y.size(0) == rows && y.size(1) == width, "fixed decay: outputs");
  DecayStep d{};
  d.f32 = is_f32(y); d.z_f32 = is_f32(z); d.z = z.data_ptr(); d.ldz = pitch(z);
  d.heads = (int)H; d.dp = (int)dp; d.vdim = (int)size[2]; d.vp = (int)vp; d.q_off = (int)size[4]; d.k_off = (int)size[5]; d.v_off = (int)size[6]; d.gate_off = (int)size[7];
  d.rows = (int)rows; d.log_decay = log_decay.data_ptr<float>(); d.state = state_ref(state, rows, H * dp * vp, "state"); d.pos = row_pos(lens, 1, rows);
  d.norm = norm.data_ptr<float>(); d.eps = (float)real[0]; d.out_scale = (float)real[1]; d.o = o.data_ptr<float>(); d.done = done.data_ptr<int>();
  d.y = y.data_ptr(); d.ldy = pitch(y);
  return d;
}
void window_step(const Tensor& z, const std::vector<int64_t>& size, const std::vector<double>& real, const Tensor& freq, const Tensor& pool, const Tensor& table,
                 const Tensor& lens, Tensor& y) {
  WindowAttn d = window_of(z, size, real, freq, pool, table, lens, 1);
  window_out(d, y, pool);
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(parallel_step(&d, nullptr, status_ptr(z), stream()));
}
void decay_step(const Tensor& z, const std::vector<int64_t>& size, const std::vector<double>& real, const Tensor& log_decay, const Tensor& state,
                const Tensor& lens, const Tensor& norm, Tensor& o, Tensor& done, Tensor& y) {
  const DecayStep d = decay_of(z, size, real, log_decay, state, lens, norm, o, done, y);
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(parallel_step(nullptr, &d, status_ptr(z), stream()));
}
// Both in one launch: y_left and y_right may be column ranges of one buffer.
void parallel_step_(const Tensor& z, const std::vector<int64_t>& wsize, const std::vector<double>& wreal, const Tensor& freq, const Tensor& pool,
                    const Tensor& table, const Tensor& lens, Tensor& y_left, const std::vector<int64_t>& dsize, const std::vector<double>& dreal,
                    const Tensor& log_decay, const Tensor& state, const Tensor& norm, Tensor& o, Tensor& done, Tensor& y_right) {
  WindowAttn w = window_of(z, wsize, wreal, freq, pool, table, lens, 1);
  window_out(w, y_left, pool);
  const DecayStep d = decay_of(z, dsize, dreal, log_decay, state, lens, norm, o, done, y_right);
  const c10::cuda::CUDAGuard guard(z.device());
  NC_CHECK(parallel_step(&w, &d, status_ptr(z), stream()));
}

std::vector<int64_t> read_status(const Tensor& like) {
  Tensor& t = status_tensor(like.device());
  const Tensor h = t.cpu();
  t.zero_();
  const int* p = h.data_ptr<int>();
  return {p[0], p[1], p[2], p[3]};
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("gemm", &gemm, py::arg("A"), py::arg("B"), py::arg("C"), py::arg("m_group") = py::none(), py::arg("epi") = 0,
        py::arg("aux") = py::none());
  m.def("attention_capped", &attention_capped);
  m.def("attention_capped_supported", &nc::attention_capped_supported);
  m.def("attention_split", &attention_split);
  m.def("attention_split_supported", &nc::attention_split_supported);
  m.def("embed_norm", &embed_norm_);
  m.def("gated_residual_norm", &gated_residual_norm_);
  m.def("poly_norm", &poly_norm_);
  m.def("layer_norm_residual", &layer_norm_residual_);
  m.def("gemv_plain", &gemv_plain, py::arg("x"), py::arg("W"), py::arg("out"), py::arg("next") = py::none());
  m.def("gemv_relu_glu", &gemv_relu_glu_, py::arg("x"), py::arg("W"), py::arg("out"), py::arg("next") = py::none());
  m.def("delta_prepare", &delta_prepare_);
  m.def("decay_prepare", &decay_prepare_);
  m.def("recurrence", &recurrence_);
  m.def("recurrence_chunks_supported", &recurrence_chunks_supported);
  m.def("recurrence_scratch", &recurrence_scratch);
  m.def("recurrence_tiles", &recurrence_tiles);
  m.def("norm_gate", &norm_gate_);
  m.def("delta_finish", &delta_finish);
  m.def("delta_step", &delta_step_);
  m.def("delta_step_supported", &delta_step_supported);
  m.def("window_post", &window_post_);
  m.def("window_attention", &window_attention_);
  m.def("window_step", &window_step);
  m.def("window_step_supported", &window_step_supported);
  m.def("decay_step", &decay_step);
  m.def("decay_step_supported", &decay_step_supported);
  m.def("parallel_step", &parallel_step_);
  m.def("latent_post", &latent_post_);
  m.def("latent_gather", &latent_gather_);
  m.def("rotate_heads", &rotate_heads_);
  m.def("absorb_query", &absorb_query_);
  m.def("latent_attention", &latent_attention_);
  m.def("latent_values", &latent_values_, py::arg("ml"), py::arg("acc"), py::arg("rows"), py::arg("heads"), py::arg("splits"), py::arg("Wuv"),
        py::arg("y"), py::arg("pdl"), py::arg("next") = py::none());
  m.def("route_topk", &route_topk_, py::arg("logits"), py::arg("experts"), py::arg("idx"), py::arg("wt"), py::arg("counts") = py::none(),
        py::arg("rank") = py::none());
  m.def("group_rows", &group_rows);
  m.def("silu_mul", &silu_mul_);
  m.def("expert_gate_up", &expert_gate_up_);
  m.def("expert_down", &expert_down_);
  m.def("expert_rows", &expert_rows_, py::arg("h"), py::arg("Wgu"), py::arg("Wdown"), py::arg("idx"), py::arg("wt"), py::arg("act"), py::arg("out"),
        py::arg("g"), py::arg("bias"), py::arg("mult"), py::arg("extra") = py::none());
  m.def("expert_rows_supported", &expert_rows_supported);
  m.def("gemv_norm", &gemv_norm, py::arg("x"), py::arg("w"), py::arg("eps"), py::arg("n"), py::arg("W"), py::arg("out"),
        py::arg("h") = py::none(), py::arg("next") = py::none());
  m.def("gemv_query_store", &gemv_query_store, py::arg("z"), py::arg("q_rank"), py::arg("q_w"), py::arg("eps"), py::arg("Wq"), py::arg("q"),
        py::arg("c_off"), py::arg("kv_rank"), py::arg("kvp"), py::arg("kv_w"), py::arg("rot_off"), py::arg("rot_dim"), py::arg("freq"),
        py::arg("pool"), py::arg("table"), py::arg("lens"), py::arg("next") = py::none());
  m.def("gemv_residual", &gemv_residual, py::arg("y"), py::arg("W"), py::arg("x"), py::arg("g"), py::arg("bias"), py::arg("mult"),
        py::arg("extra") = py::none(), py::arg("next") = py::none(), py::arg("accumulate") = true, py::arg("pdl") = true);
  m.def("read_status", &read_status);
  m.def("launch_count", [] { return g_launches.load(); });
}
