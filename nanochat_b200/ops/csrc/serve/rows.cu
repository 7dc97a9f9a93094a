// Row kernels of the serving path.
//
//   embed_norm            token embedding into the float residual stream, and its norm
//   gated_residual_norm   residual update by sigmoid-gated sublayer outputs (a mixture of experts' weighted rows are
//                         summed on the way in), then the next norm: one pass, the row stays in registers / L1
//   poly_norm             the normed-powers activation
//   gemv                  matrix-vector products of a decode step with the work around them folded in: the norm or the
//                         activation of the input (both enter linearly once the row statistics are known, so the
//                         statistics ride along with the dot products), the gated residual update of the output, and
//                         extra CTAs that append the step's entry to the latent store
// One CTA per row for the first three. gemv: a CTA owns four outputs and its 256 threads split K.
#include "latent_store.cuh"

namespace nc {
namespace serve {

namespace {

template <typename T>
__global__ void __launch_bounds__(256)
embed_norm_kernel(const long long* __restrict__ ids, const T* __restrict__ table, long long ld, int vocab,
                  const float* __restrict__ w, float eps, int n, int np, float* __restrict__ x, float* __restrict__ x0,
                  T* __restrict__ h) {
  __shared__ float red[32];
  const long long row = blockIdx.x;
  pdl_wait();
  pdl_trigger();
  long long id = ids[row];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + id * ld;
  float ss[1] = {0.f};
  for (int c = threadIdx.x * 8; c < np; c += blockDim.x * 8) {
    float v[8];
    load8(src + c, v);
    store8(x + row * np + c, v);
    if (x0) store8(x0 + row * np + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss[0] += v[j] * v[j];
  }
  if (h == nullptr) return;
  block_sum<1>(ss, red);
  const float r = inv_rms(ss[0], n, eps);
  for (int c = threadIdx.x * 8; c < np; c += blockDim.x * 8) {
    float v[8], wv[8];
    load8(src + c, v);
    load8(w + c, wv);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= r * wv[j];
    store8(h + row * np + c, v);
  }
}

struct TermsT { GatedTerm t[2]; int n; };

template <typename T>
__global__ void __launch_bounds__(256)
gated_residual_norm_kernel(float* __restrict__ x, TermsT terms, float mult, const float* __restrict__ extra,
                           const float* __restrict__ w, float eps, int n, int np, T* __restrict__ h) {
  __shared__ float red[32];
  const long long row = blockIdx.x;
  float ss[1] = {0.f};
  for (int c = threadIdx.x * 8; c < np; c += blockDim.x * 8) {
    float v[8], sum[8];
    load8(x + row * np + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) sum[j] = 0.f;
    for (int t = 0; t < terms.n; ++t) {
      const GatedTerm& g = terms.t[t];
      float gv[8], bv[8], y[8];
      load8((const T*)g.g + row * g.ldg + c, gv);
      load8(g.bias + c, bv);
      if (g.slot == nullptr) {
        load8((const T*)g.y + row * g.ldy + c, y);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) y[j] = 0.f;
        for (int k = 0; k < g.top; ++k) {
          float e[8];
          load8((const T*)g.y + (long long)g.slot[row * g.top + k] * g.ldy + c, e);
          const float wt = g.wt[row * g.top + k];
#pragma unroll
          for (int j = 0; j < 8; ++j) y[j] += wt * e[j];
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) sum[j] += sigmoidf(gv[j] + bv[j]) * y[j];
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] += mult * sum[j];
    if (extra) {
      float e[8];
      load8(extra + row * np + c, e);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] += e[j];
    }
    store8(x + row * np + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss[0] += v[j] * v[j];
  }
  block_sum<1>(ss, red);
  const float r = inv_rms(ss[0], n, eps);
  for (int c = threadIdx.x * 8; c < np; c += blockDim.x * 8) {        // a thread re-reads what it wrote itself
    float v[8], wv[8];
    load8(x + row * np + c, v);
    load8(w + c, wv);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= r * wv[j];
    store8(h + row * np + c, v);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
poly_norm_kernel(const T* __restrict__ z, long long ldz, const float* __restrict__ coef, float eps, int n, int np,
                 T* __restrict__ out, long long ldo) {
  __shared__ float red[96];
  const long long row = blockIdx.x;
  const T* src = z + row * ldz;
  float ss[3] = {0.f, 0.f, 0.f};
  for (int c = threadIdx.x * 8; c < np; c += blockDim.x * 8) {
    float v[8];
    load8(src + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c + j < n) { const float q = v[j] * v[j]; ss[0] += q; ss[1] += q * q; ss[2] += q * q * q; }
    }
  }
  block_sum<3>(ss, red);
  const float a = coef[0] * inv_rms(ss[0], n, eps), b = coef[1] * inv_rms(ss[1], n, eps), d = coef[2] * inv_rms(ss[2], n, eps);
  const float e = coef[3];
  for (int c = threadIdx.x * 8; c < np; c += blockDim.x * 8) {
    float v[8];
    load8(src + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = c + j < n ? v[j] * (a + v[j] * (b + v[j] * d)) + e : 0.f;
    store8(out + row * ldo + c, v);
  }
}

// ------------------------------------------------------------------------------- gemv
constexpr int COLS = 4;        // outputs per CTA

struct GemvArgs {
  const void* x; long long ldx;
  const float* w; float eps; int n_real;
  const bf16* W; long long ldw;
  int N, K, epi;
  void* out; long long ldo;
  float* resid; long long ldr; const float* g; long long ldg; const float* bias; float mult; const float* extra;
  bf16* h_out; long long ldh;
  NextWeights next;
  LatentStore store;
  int n_blocks;
};

template <int B, int PRE>
__global__ void __launch_bounds__(256)
gemv_kernel(const GemvArgs a) {
  constexpr int KINDS = PRE == PRE_POLY ? 3 : 1;
  constexpr int SS = PRE == PRE_POLY ? 3 : 1;
  __shared__ float s_acc[8][KINDS][COLS][B];
  __shared__ float s_w[8][COLS];
  __shared__ float s_ss[8][SS][B];
  __shared__ float s_red[32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (PRE == PRE_NORM && (int)blockIdx.x >= a.n_blocks) {              // extra CTAs: append to the latent store
    const int b = blockIdx.x - a.n_blocks;
    pdl_wait();
    pdl_trigger();
    const LatentStore& d = a.store;
    const int pos = d.pos.lens[b / d.pos.per_seq] + b % d.pos.per_seq;
    const long long off = token_offset(d.pg, b / d.pos.per_seq, pos);
    if (off < 0) {
      if (tid == 0 && d.status) atomicCAS(d.status, 0, (ST_BAD_ARG << 24) | 0x57043);
      return;
    }
    const float* z = (const float*)d.z + (long long)b * d.ldz;
    store_latent<bf16, float>(z, z + d.rot_off, d.kv_rank, d.kvp, d.kv_w, d.eps, d.rot_dim, d.rp, d.dims, d.freq, pos,
                              (bf16*)d.pg.pool + off, (bf16*)nullptr, s_red);
    return;
  }
  const int n0 = blockIdx.x * COLS;
  float acc[KINDS][COLS][B], ss[SS][B], wsum[COLS];
#pragma unroll
  for (int b = 0; b < B; ++b) {
#pragma unroll
    for (int q = 0; q < SS; ++q) ss[q][b] = 0.f;
#pragma unroll
    for (int q = 0; q < KINDS; ++q)
#pragma unroll
      for (int r = 0; r < COLS; ++r) acc[q][r][b] = 0.f;
  }
#pragma unroll
  for (int r = 0; r < COLS; ++r) wsum[r] = 0.f;
  prefetch_l2_slice(a.next, blockIdx.x, a.n_blocks);
  const int k_first = tid * 8;
  uint4 pre[COLS];
#pragma unroll
  for (int r = 0; r < COLS; ++r)
    pre[r] = k_first < a.K ? ld_once(a.W + (long long)min(n0 + r, a.N - 1) * a.ldw + k_first) : make_uint4(0, 0, 0, 0);
  pdl_wait();
  pdl_trigger();
  auto chunk = [&](const uint4 (&wv)[COLS], int k) {
    float wf[COLS][8], nw[8];
#pragma unroll
    for (int r = 0; r < COLS; ++r) unpack8(wv[r], wf[r]);
    if (PRE == PRE_NORM) load8(a.w + k, nw);
    if (PRE == PRE_POLY) {
#pragma unroll
      for (int r = 0; r < COLS; ++r)
#pragma unroll
        for (int j = 0; j < 8; ++j) wsum[r] += wf[r][j];
    }
#pragma unroll
    for (int b = 0; b < B; ++b) {
      float xf[8];
      if (PRE == PRE_PLAIN) load8((const bf16*)a.x + b * a.ldx + k, xf);
      else load8((const float*)a.x + b * a.ldx + k, xf);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (PRE == PRE_NORM) { ss[0][b] += xf[j] * xf[j]; xf[j] *= nw[j]; }
        if (PRE == PRE_POLY) {
          const float q = xf[j] * xf[j];
          ss[0][b] += q; ss[1 % SS][b] += q * q; ss[2 % SS][b] += q * q * q;
          const float q3 = q * xf[j];
#pragma unroll
          for (int r = 0; r < COLS; ++r) {
            acc[0][r][b] += wf[r][j] * xf[j];
            acc[1 % KINDS][r][b] += wf[r][j] * q;
            acc[2 % KINDS][r][b] += wf[r][j] * q3;
          }
        } else {
#pragma unroll
          for (int r = 0; r < COLS; ++r) acc[0][r][b] += wf[r][j] * xf[j];
        }
      }
    }
  };
  if (k_first < a.K) chunk(pre, k_first);
#pragma unroll 2
  for (int k = k_first + 2048; k < a.K; k += 2048) {
    uint4 wv[COLS];
#pragma unroll
    for (int r = 0; r < COLS; ++r) wv[r] = ld_once(a.W + (long long)min(n0 + r, a.N - 1) * a.ldw + k);
    chunk(wv, k);
  }
  {
    constexpr int NV = pow2_ceil(COLS * B), LOW = 5 - ilog2(NV);
#pragma unroll
    for (int q = 0; q < KINDS; ++q) {
      float flat[NV];
#pragma unroll
      for (int i = 0; i < NV; ++i) flat[i] = i < COLS * B ? acc[q][i / B][i % B] : 0.f;
      const float total = warp_sum_many<NV>(flat, lane);
      const int idx = lane >> LOW;
      if ((lane & ((1 << LOW) - 1)) == 0 && idx < COLS * B) s_acc[warp][q][idx / B][idx % B] = total;
    }
  }
  if (PRE != PRE_PLAIN) {
    constexpr int NB = pow2_ceil(B), LOW = 5 - ilog2(NB);
#pragma unroll
    for (int q = 0; q < SS; ++q) {
      float flat[NB];
#pragma unroll
      for (int i = 0; i < NB; ++i) flat[i] = i < B ? ss[q][i] : 0.f;
      const float total = warp_sum_many<NB>(flat, lane);
      const int idx = lane >> LOW;
      if ((lane & ((1 << LOW) - 1)) == 0 && idx < B) s_ss[warp][q][idx] = total;
    }
  }
  if (PRE == PRE_POLY) {
    const float total = warp_sum_many<COLS>(wsum, lane);
    if ((lane & 7) == 0) s_w[warp][lane >> 3] = total;
  }
  __syncthreads();
  auto stat = [&](int q, int b) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) t += s_ss[w][q][b];
    return inv_rms(t, a.n_real, a.eps);
  };
  if (PRE == PRE_NORM && a.h_out != nullptr && blockIdx.x == 0) {
    for (int b = 0; b < B; ++b) {
      const float r = stat(0, b);
      for (int k = tid * 8; k < a.K; k += 2048) {
        float xf[8], nw[8];
        load8((const float*)a.x + b * a.ldx + k, xf);
        load8(a.w + k, nw);
#pragma unroll
        for (int j = 0; j < 8; ++j) xf[j] *= r * nw[j];
        store8(a.h_out + b * a.ldh + k, xf);
      }
    }
  }
  if (tid < COLS * B) {
    const int r = tid / B, b = tid - r * B;
    const int n = n0 + r;
    if (n < a.N) {
      float v[KINDS];
#pragma unroll
      for (int q = 0; q < KINDS; ++q) {
        v[q] = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v[q] += s_acc[w][q][r][b];
      }
      float o = v[0];
      if (PRE == PRE_NORM) o *= stat(0, b);
      if (PRE == PRE_POLY) {
        float sw = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) sw += s_w[w][r];
        o = a.w[0] * stat(0, b) * v[0] + a.w[1] * stat(1 % SS, b) * v[1 % KINDS] + a.w[2] * stat(2 % SS, b) * v[2 % KINDS] +
            a.w[3] * sw;
      }
      if (a.epi == GEMV_STORE_F32) {
        ((float*)a.out)[b * a.ldo + n] = o;
      } else if (a.epi == GEMV_STORE_BF16) {
        ((bf16*)a.out)[b * a.ldo + n] = __float2bfloat16_rn(o);
      } else {
        float x = a.resid[b * a.ldr + n] + a.mult * sigmoidf(a.g[b * a.ldg + n] + a.bias[n]) * o;
        if (a.extra) x += a.extra[b * a.ldr + n];
        a.resid[b * a.ldr + n] = x;
      }
    }
  }
}

}  // namespace

cudaError_t embed_norm(bool f32, const long long* ids, const void* table, long long ld, int vocab, const float* w,
                       float eps, int rows, int n, int np, float* x, float* x0, void* h, cudaStream_t s) {
  if (rows <= 0 || n <= 0 || n > np || (np & 7) || (ld & 7) || ld < np || vocab <= 0) return cudaErrorInvalidValue;
  if (f32)
    return launch_pdl(embed_norm_kernel<float>, dim3(rows), dim3(256), 0, s, ids, (const float*)table, ld, vocab, w, eps, n, np, x, x0, (float*)h);
  return launch_pdl(embed_norm_kernel<bf16>, dim3(rows), dim3(256), 0, s, ids, (const bf16*)table, ld, vocab, w, eps, n, np, x, x0, (bf16*)h);
}

cudaError_t gated_residual_norm(bool f32, float* x, const GatedTerm* terms, int n_terms, float mult, const float* extra,
                                const float* w, float eps, int rows, int n, int np, void* h, cudaStream_t s) {
  if (rows <= 0 || n <= 0 || n > np || (np & 7) || n_terms < 0 || n_terms > 2) return cudaErrorInvalidValue;
  TermsT t{};
  t.n = n_terms;
  for (int i = 0; i < n_terms; ++i) {
    if ((terms[i].ldg & 7) || (terms[i].ldy & 7)) return cudaErrorInvalidValue;
    t.t[i] = terms[i];
  }
  if (f32) gated_residual_norm_kernel<float><<<rows, 256, 0, s>>>(x, t, mult, extra, w, eps, n, np, (float*)h);
  else gated_residual_norm_kernel<bf16><<<rows, 256, 0, s>>>(x, t, mult, extra, w, eps, n, np, (bf16*)h);
  return cudaGetLastError();
}

cudaError_t poly_norm(bool f32, const void* z, long long ldz, const float* coef, float eps, int rows, int n, int np,
                      void* out, long long ldo, cudaStream_t s) {
  if (rows <= 0 || n <= 0 || n > np || (np & 7) || (ldz & 7) || (ldo & 7)) return cudaErrorInvalidValue;
  if (f32) poly_norm_kernel<float><<<rows, 256, 0, s>>>((const float*)z, ldz, coef, eps, n, np, (float*)out, ldo);
  else poly_norm_kernel<bf16><<<rows, 256, 0, s>>>((const bf16*)z, ldz, coef, eps, n, np, (bf16*)out, ldo);
  return cudaGetLastError();
}

template <int PRE>
static cudaError_t gemv_rows(int rows, const GemvArgs& a, int grid, cudaStream_t s) {
  switch (rows) {
#define NC_G(B) case B: return launch_pdl(gemv_kernel<B, PRE>, dim3(grid), dim3(256), 0, s, a);
    NC_G(1) NC_G(2) NC_G(3) NC_G(4) NC_G(5) NC_G(6) NC_G(7) NC_G(8)
#undef NC_G
  }
  return cudaErrorInvalidValue;
}

cudaError_t gemv(const GemvDesc& d, int pre, int epi, cudaStream_t s) {
  if (d.rows < 1 || d.rows > 8 || d.N <= 0 || d.K <= 0 || (d.K & 7) || (d.ldx & 7) || (d.ldw & 7) || d.n_real > d.K)
    return cudaErrorInvalidValue;
  if (pre != PRE_PLAIN && (d.w == nullptr || d.n_real <= 0)) return cudaErrorInvalidValue;
  if (epi == GEMV_RESIDUAL ? (d.resid == nullptr || d.g == nullptr || d.bias == nullptr) : d.out == nullptr)
    return cudaErrorInvalidValue;
  if (d.store != nullptr && pre != PRE_NORM) return cudaErrorInvalidValue;
  if (d.h_out != nullptr && (pre != PRE_NORM || (d.ldh & 7))) return cudaErrorInvalidValue;
  GemvArgs a{};
  a.x = d.x; a.ldx = d.ldx; a.w = d.w; a.eps = d.eps; a.n_real = d.n_real;
  a.W = (const bf16*)d.W; a.ldw = d.ldw; a.N = d.N; a.K = d.K; a.epi = epi;
  a.out = d.out; a.ldo = d.ldo; a.resid = d.resid; a.ldr = d.ldr; a.g = d.g; a.ldg = d.ldg; a.bias = d.bias;
  a.mult = d.mult; a.extra = d.extra; a.h_out = (bf16*)d.h_out; a.ldh = d.ldh; a.next = d.next;
  a.n_blocks = (d.N + COLS - 1) / COLS;
  int grid = a.n_blocks;
  if (d.store) { a.store = *d.store; grid += d.rows; }
  if (pre == PRE_NORM) return gemv_rows<PRE_NORM>(d.rows, a, grid, s);
  if (pre == PRE_PLAIN) return gemv_rows<PRE_PLAIN>(d.rows, a, grid, s);
  if (pre == PRE_POLY) return gemv_rows<PRE_POLY>(d.rows, a, grid, s);
  return cudaErrorInvalidValue;
}

}  // namespace serve
}  // namespace nc
