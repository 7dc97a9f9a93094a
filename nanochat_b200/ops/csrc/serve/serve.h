// Host interface of the serving kernels: rows.cu (norms, residual updates, activations), gemv.cu (matrix-vector products of
// a decode step), latent.cu (latent attention over a paged store), experts.cu (mixture of experts), window.cu (window
// attention whose values are its unrotated keys), recurrent.cu (gated delta rule, linear attention with a fixed decay) and
// step.cu (one token of the last two per row).
//
// Conventions. "f32" selects float or bf16 for the typed pointers (weights and activations share one type). The
// residual stream, gates' biases, norm weights, router logits and attention partials are always float. Row sizes and
// pitches are multiples of 8 elements, pointers 16-byte aligned; entries past a row's real size are zero.
#pragma once

#include <cuda_runtime.h>
#include <stddef.h>

namespace nc {
namespace serve {

// One layer's paged store: n_pages pages of 2^shift tokens, each token `width` elements; `table` (sequences x
// max_pages) names the page of every 2^shift tokens of a sequence.
struct Pages {
  void* pool;
  const int* table;
  int max_pages, shift, n_pages, width;
};

// Rows of a step: row r belongs to sequence r / per_seq and sits at position lens[r / per_seq] + r % per_seq.
struct RowPos {
  const int* lens;
  int per_seq;
};

struct NextWeights {      // memory a later kernel will stream; ptr = nullptr: none
  const void* ptr;
  long long bytes;
};

// ------------------------------------------------------------------------------ rows.cu
// x[r] = table[ids[r]] (float), x0[r] the same when x0 is given, h[r] = x / rms(x) * w. Ids are clamped to [0, vocab).
cudaError_t embed_norm(bool f32, const long long* ids, const void* table, long long ld, int vocab, const float* w,
                       float eps, int rows, int n, int np, float* x, float* x0, void* h, cudaStream_t s);

// One term of the residual update: sigmoid(g + bias) * y, y a row or the weighted sum of the rows a token's experts
// wrote (slot / wt: rows x top).
struct GatedTerm {
  const void* g; long long ldg;
  const float* bias;
  const void* y; long long ldy;
  const int* slot; const float* wt; int top;
};
// x[r] += mult * sum of terms (+ extra[r]); h[r] = x / rms(x) * w.
cudaError_t gated_residual_norm(bool f32, float* x, const GatedTerm* terms, int n_terms, float mult, const float* extra,
                                const float* w, float eps, int rows, int n, int np, void* h, cudaStream_t s);

// x[r] += N(y[r]) * wy; h[r] = N(x[r]) * w, N the layer norm (mean removed) over the row's n entries. With ids given the
// stream opens: x[r] = N(y[ids[r]]) * wy, ids clamped to [0, vocab). Rows of up to 8192 entries.
cudaError_t layer_norm_residual(bool f32, bool y_f32, const long long* ids, const void* y, long long ldy, int vocab, const float* wy, float* x,
                                const float* w, float eps, int rows, int n, int np, void* h, cudaStream_t s);

// out[r] = c[0] N(z) + c[1] N(z^2) + c[2] N(z^3) + c[3], N(v) = v / rms(v) over the row's n entries.
cudaError_t poly_norm(bool f32, bool z_f32, const void* z, long long ldz, const float* coef, float eps, int rows, int n, int np,
                      void* out, long long ldo, cudaStream_t s);

// ------------------------------------------------------------------------------ gemv.cu
// Matrix-vector products of a decode step, bf16 weights, rows <= 8 (plain stores: any number, eight at a time; for few outputs): out[b, j] = epilogue(sum_k pre(x)[b, k] W[j, k]).
enum GemvPre : int {
  PRE_NORM = 0,     // x float, x / rms(x) * w
  PRE_PLAIN = 1,    // x bf16
};
enum GemvEpi : int {
  GEMV_STORE_F32 = 0,
  GEMV_STORE_BF16 = 1,
  GEMV_RESIDUAL = 2,     // resid[b, j] (+)= mult * sigmoid(g[b, j] + bias[j]) * value (+ extra[b, j])
};
struct LatentStore {     // see latent_store below; used by the extra CTAs of a product that also appends to the store
  const void* z; long long ldz;
  int kv_rank, kvp; const float* kv_w; float eps;
  int rot_off, rot_dim, rp, dims; const float* freq;
  Pages pg; RowPos pos; int* status;
};
struct GemvDesc {
  const void* x; long long ldx;
  const float* w; float eps; int n_real;            // norm weight, entries of the row that count
  const void* W; long long ldw;
  int rows, N, K;
  void* out; long long ldo;
  float* resid; long long ldr; const float* g; long long ldg; const float* bias; float mult; const float* extra;
  bool accumulate;                                  // GEMV_RESIDUAL: add to resid, or overwrite it
  void* h_out; long long ldh;                       // PRE_NORM: the normed row as bf16, when wanted
  NextWeights next;
  const LatentStore* store;                         // PRE_NORM only
  bool pdl;
};
cudaError_t gemv(const GemvDesc& d, int pre, int epi, cudaStream_t s);
// out[b, j] = relu(x[b] . W[j]) * (x[b] . W[N + j]), bf16: W holds N gate rows, then N up rows (PRE_PLAIN fields of d)
cudaError_t gemv_relu_glu(const GemvDesc& d, cudaStream_t s);
// The experts of a decode step, rows <= 8: out[b] = mult * sigmoid(g + bias) * sum_k wt[b, k] expert(idx[b, k])(h[b]) (+ extra).
// act: rows * top x fp scratch.
struct ExpertRows {
  const void* h; long long ldh; int rows, top, experts, K, fp, N;
  const void* Wgu; const void* Wdown;
  const int* idx; const float* wt;
  void* act;
  float* out; long long ldo; const float* g; long long ldg; const float* bias; float mult; const float* extra;
};
bool expert_rows_supported(int rows, int top);
cudaError_t expert_rows(const ExpertRows& d, cudaStream_t s);

// ---------------------------------------------------------------------------- latent.cu
// Per row: cq = norm(z[:q_rank]) (when asked), and the entry [norm(z[c_off:c_off+kv_rank]) | rotated z[rot_off:]]
// into the store and (kv_out) a dense row. TZ of z: float when z_f32.
struct LatentPost {
  bool f32, z_f32;
  const void* z; long long ldz; int rows;
  int q_rank, qp; const float* q_w; void* cq; long long ldcq;
  int c_off, kv_rank, kvp; const float* kv_w; float eps;
  int rot_off, rot_dim, rp, dims; const float* freq;
  Pages pg; RowPos pos;
  void* kv_out; long long ldkv;
};
cudaError_t latent_post(const LatentPost& d, int* status, cudaStream_t s);
// out[j] = the store's entry of token first + j of sequence `seq`, j < count.
cudaError_t latent_gather(bool f32, const Pages& pg, int seq, int first, int count, void* out, long long ldo,
                          int* status, cudaStream_t s);
// q[r, h, off : off + dims] rotated in place (rows x heads x head_pitch).
cudaError_t rotate_heads(bool f32, void* q, long long ldq, int rows, int heads, int head_pitch, int off, int dims,
                         const float* freq, const RowPos& pos, cudaStream_t s);
// qa[r, h, :] = sum_d q[r, h, d] Wuk[h * dp + d, :]     (d < dp)
cudaError_t absorb_query(bool f32, const void* q, long long ldq, int rows, int heads, int head_pitch, int dp,
                         const void* Wuk, int kvp, void* qa, bool pdl, cudaStream_t s);
// Attention of absorbed queries over stored entries; per (row, head, split) an unnormalised partial
// [max, sum] in ml and sum of exp weights times latents in acc (kvp floats). The query's last part is rotated here.
struct LatentAttn {
  bool f32;
  const void* qa; const void* q; long long ldq; int head_pitch, dp, rot_dim, rp, dims; const float* freq;
  int rows, heads, kvp;
  Pages pg; RowPos pos;
  int window;            // keys a query sees, itself included; <= 0: all
  float scale;
  int splits;
  float* ml; float* acc;
  bool pdl;
};
cudaError_t latent_attention(const LatentAttn& d, cudaStream_t s);
bool latent_attention_tensor_cores(const LatentAttn& d);
// y[r, h * vp + j] = sum_k merged(r, h)[k] Wuv[h * vp + j, k], merged = the splits' partials combined and normalised.
cudaError_t latent_values(bool f32, const float* ml, const float* acc, int rows, int heads, int splits, int kvp,
                          const void* Wuv, int vp, void* y, long long ldy, bool pdl, const NextWeights& next,
                          cudaStream_t s);

// --------------------------------------------------------------------------- experts.cu
// The `top` largest logits of every row (ties: lower index first) and the softmax over them. counts / rank (optional):
// how many rows chose an expert, and a row's place among them.
cudaError_t route_topk(const float* logits, long long ld, int rows, int experts, int top, int* idx, float* wt,
                       int* counts, int* rank, cudaStream_t s);
// Rows grouped by expert, every group starting at a multiple of 128: offsets (experts), tile_group (tiles, -1 = unused).
cudaError_t plan_groups(const int* counts, int experts, int* offsets, int* tile_group, int tiles, cudaStream_t s);
// xg[slot] = h[r], slot[r, k] = offsets[idx[r, k]] + rank[r, k]
cudaError_t gather_groups(const void* h, long long ldh, int rows, int top, int np, const int* idx, const int* rank,
                          const int* offsets, int* slot, void* xg, cudaStream_t s);
// act[i, :fp] = silu(gu[i, :fp]) * gu[i, fp:2fp] for the rows of used tiles (bf16)
cudaError_t silu_mul(const void* gu, int rows, int fp, const int* tile_group, void* act, cudaStream_t s);

// Experts as matrix-vector products, one per (row, chosen expert). Wgu: experts x [gate fp rows | up fp rows] x K.
struct Routing {
  const int* idx; const float* wt;      // rows x top
  int experts, top;
};
cudaError_t expert_gate_up(bool f32, const void* h, long long ldh, int rows, int K, const void* Wgu, int fp,
                           const Routing& rt, void* act, cudaStream_t s);
// y[r] = sum_k wt[r, k] Wdown[idx[r, k]] act[r * top + k]
struct ExpertDown {
  bool f32;
  const void* act; int rows, fp;
  const void* Wdown; int N;
  Routing rt;
  void* y; long long ldy;
};
cudaError_t expert_down(const ExpertDown& d, cudaStream_t s);

// ---------------------------------------------------------------------------- window.cu
// Window attention with grouped keys that also serve as values: entry of a token in the store = [kv_heads x dp rotated
// keys | kv_heads x dp keys as projected]. Rotation pairs entries 2i and 2i + 1 of the first `dims`. Scores are
// softcap * tanh(scale q.k / softcap) (softcap <= 0: no cap); y is multiplied by out_scale. freq: dims / 2 frequencies,
// then what their floats leave over.
struct WindowAttn {
  bool f32, z_f32;
  const void* z; long long ldz;           // queries at q_off (heads x dp), keys at k_off (kv_heads x dp)
  int q_off, k_off;
  int rows, heads, kv_heads, dp, dims; const float* freq;
  Pages pg; RowPos pos;
  int window;                             // keys a query sees, itself included; <= 0: all
  float scale, softcap, out_scale;
  void* y; long long ldy;                 // rows x (heads x dp)
};
// Queries rotated in place, the rows' entries into the store and (dense) a dense row.
cudaError_t window_post(const WindowAttn& d, void* dense, long long ldd, int* status, cudaStream_t s);
// Plain form for any size: rotated queries in z against the store, which holds the rows' own entries already.
cudaError_t window_attention(const WindowAttn& d, cudaStream_t s);

// ------------------------------------------------------------------------- recurrent.cu
// Two recurrences over a per-sequence state S (heads x dp x vp floats):
//   delta    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q      unit keys and queries, g and beta per token
//   decay    S <- decay_h S + k v^T;           o = S^T q
// A sequence at position 0 starts from zeros whatever its state memory holds.
struct StateRef {
  float* ptr; long long seq_stride;       // floats between sequences
};
// Inputs of the delta rule: q and k of kv_heads heads, v of heads heads, as projected, side by side in z (channels
// [0, 2 kv_heads dp + heads vp)); a causal convolution of `taps` per channel and silu come first. The ring keeps the inputs
// of the last taps - 1 tokens per channel: token t in slot t % taps.
struct DeltaInputs {
  bool f32, z_f32;
  const void* z; long long ldz;
  int rows, heads, kv_heads, dim, dp, vdim, vp, taps;
  const float* conv;                      // taps x channels, the last row meets the current token
  const float* ba; long long ldba; int a_off;   // per row: heads logits of beta, at a_off heads inputs of the decay
  const float* neg_a; const float* dt_bias;     // log g = neg_a * softplus(a + dt_bias)
  StateRef ring;
  RowPos pos;
};
// Convolution and silu of every channel into out: rows x channels, or (tiles, bf16) recurrence_tiles() bytes for
// recurrence_chunks; norms (rows x 2 kv_heads) = 1 / |q| * dim^-1/2, then 1 / |k|; beta_g (rows x 2 heads) = beta, then log g.
cudaError_t delta_prepare(const DeltaInputs& d, bool tiles, void* out, float* norms, float* beta_g, cudaStream_t s);
// silu of q, k (heads x dp each) and v (heads x vp), side by side in z, into out likewise.
cudaError_t decay_prepare(bool f32, const void* z, long long ldz, int rows, int per_seq, int heads, int dp, int vp, bool tiles, void* out, cudaStream_t s);

struct Recurrence {
  bool f32;
  const void* act; long long lda;         // rows: q at q_off, k at k_off (kv_heads x dp), v at v_off (heads x vp)
  int q_off, k_off, v_off;
  int rows, heads, kv_heads, dp, vp;
  const float* norms; const float* beta_g;      // delta rule
  const float* log_decay;                       // fixed decay: natural logarithm per head (beta_g == nullptr)
  StateRef state;
  RowPos pos;
  void* o; long long ldo;                 // rows x (heads x vp)
};
// Token by token; any T, float or bf16, dp <= 512.
cudaError_t recurrence_scan(const Recurrence& d, cudaStream_t s);
// Chunks of 64 tokens on the tensor cores, bf16, dp <= 128: act holds tiles (lda and offsets unused), scratch
// recurrence_scratch() bytes.
bool recurrence_chunks_supported(int dp);
size_t recurrence_tiles(int seqs, int per_seq, int heads, int kv_heads, int dp, int vp);
size_t recurrence_scratch(int seqs, int per_seq, int heads, bool delta);
cudaError_t recurrence_chunks(const Recurrence& d, void* scratch, int* status, cudaStream_t s);

// y = o / rms(o) * w * act(gate) * out_scale; groups of np entries (n real ones) are normed apart, w (np) is shared by the
// groups. act: 0 silu, 1 sigmoid. ring (optional, delta): also keep the last inputs of the rows' convolution.
cudaError_t norm_gate(bool f32, const void* o, long long ldo, const void* gate, long long ldg, const float* w, float eps, int rows, int groups,
                      int n, int np, int act, float out_scale, void* y, long long ldy, const DeltaInputs* ring, cudaStream_t s);

// ------------------------------------------------------------------------------ step.cu
// One token per row (RowPos::per_seq == 1).
// Delta rule from z to y (rows x (heads x vp), bf16 or float), state and ring updated, norm and silu gate included.
struct DeltaStep {
  DeltaInputs in;
  StateRef state;
  const float* norm; float eps;
  int gate_off;                           // gate logits in z (heads x vp)
  void* y; long long ldy;
};
bool delta_step_supported(int dp, int vp);
cudaError_t delta_step(const DeltaStep& d, cudaStream_t s);
// Fixed decay from z to y: q, k, v, gate logits side by side at q_off, k_off, v_off, gate_off of z.
struct DecayStep {
  bool f32, z_f32;
  const void* z; long long ldz;
  int q_off, k_off, v_off, gate_off;
  int rows, heads, dp, vp, vdim;
  const float* log_decay;
  StateRef state;
  RowPos pos;
  const float* norm; float eps, out_scale;
  float* o;                               // rows x (heads x vp) scratch
  int* done;                              // rows counters, zero before and after
  void* y; long long ldy;
};
bool decay_step_supported(int dp, int vp);
// Either mechanism or both side by side in one launch; attention (bf16) appends the token's entry to the store itself.
bool window_step_supported(bool f32, int dp);
cudaError_t parallel_step(const WindowAttn* left, const DecayStep* right, int* status, cudaStream_t s);

}  // namespace serve
}  // namespace nc
