// Row kernels of the serving path.
//
//   embed_norm            token embedding into the float residual stream, and its norm
//   gated_residual_norm   residual update by sigmoid-gated sublayer outputs (a mixture of experts' weighted rows are
//                         summed on the way in), then the next norm: one pass, the row stays in registers / L1
//   layer_norm_residual   a sublayer's output normed, added to the residual stream, and the next sublayer's norm; the same
//                         with a token's embedding in place of the sublayer opens the stream
//   poly_norm             the normed-powers activation
// One CTA per row.
#include "common.cuh"

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
__global__ void __launch_bounds__(256, 4)
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
      for (int j = 0; j < 8; ++j) sum[j] += sigmoid_of<T>(gv[j] + bv[j]) * y[j];
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

// A row of np <= 8 * THREADS * NV entries sits in the registers of a block: entry (i * THREADS + threadIdx.x) * 8 + j.
template <int THREADS, int NV, typename TY>
__device__ __forceinline__ void load_row(float (&v)[NV][8], const TY* src, int np) {
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * THREADS + threadIdx.x) * 8;
    if (c < np) {
      load8(src + c, v[i]);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = 0.f;
    }
  }
}
// Sum over the block with one barrier; `red` (THREADS / 32 floats) is used by this call alone.
template <int THREADS>
__device__ __forceinline__ float row_sum(float s, float* red) {
  constexpr int WARPS = THREADS / 32;
  s = warp_sum(s);
  const int lane = threadIdx.x & 31;
  if (lane == 0) red[threadIdx.x >> 5] = s;
  __syncthreads();
  s = 0.f;
#pragma unroll
  for (int w = 0; w < WARPS; w += 4) {
    const float4 t = *reinterpret_cast<const float4*>(red + w);
    s += (t.x + t.y) + (t.z + t.w);
  }
  return s;
}
// v = (v - mean) / sqrt(variance + eps) * w over the first n entries; v and w are zero past them. red: two sums' memory.
template <int THREADS, int NV>
__device__ __forceinline__ void layer_norm_row(float (&v)[NV][8], const float (&w)[NV][8], int n, float eps, float* red) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) s += v[i][j];
  const float mean = row_sum<THREADS>(s, red) / n;
  s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int left = n - (i * THREADS + (int)threadIdx.x) * 8;      // entries of this vector that count
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      v[i][j] -= mean;
      if (j < left) s += v[i][j] * v[i][j];
    }
  }
  const float r = inv_rms(row_sum<THREADS>(s, red + 8), n, eps);
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) v[i][j] *= r * w[i][j];
}

// T: type of h; TY: type of y (an embedding table's rows when ids is given)
template <typename T, typename TY, int THREADS, int NV>
__global__ void __launch_bounds__(THREADS)
layer_norm_residual_kernel(const long long* __restrict__ ids, const TY* __restrict__ y, long long ldy, int vocab, const float* __restrict__ wy,
                           float* __restrict__ x, const float* __restrict__ w, float eps, int n, int np, T* __restrict__ h) {
  __shared__ __align__(16) float red[4][8];
  const long long row = blockIdx.x;
  float wv[NV][8], v[NV][8], xv[NV][8];
  load_row<THREADS, NV>(wv, wy, np);
  pdl_wait();
  pdl_trigger();
  long long src = row;
  if (ids != nullptr) {
    src = ids[row];
    src = src < 0 ? 0 : (src >= vocab ? vocab - 1 : src);
  }
  load_row<THREADS, NV>(v, y + src * ldy, np);
  if (ids == nullptr) load_row<THREADS, NV>(xv, (const float*)x + row * np, np);
  layer_norm_row<THREADS, NV>(v, wv, n, eps, red[0]);
  load_row<THREADS, NV>(wv, w, np);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * THREADS + threadIdx.x) * 8;
    if (ids == nullptr) {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] += xv[i][j];
    }
    if (c < np) store8(x + row * np + c, v[i]);
  }
  layer_norm_row<THREADS, NV>(v, wv, n, eps, red[2]);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * THREADS + threadIdx.x) * 8;
    if (c < np) store8(h + row * np + c, v[i]);
  }
}

template <typename T, typename TZ>
__global__ void __launch_bounds__(256)
poly_norm_kernel(const TZ* __restrict__ z, long long ldz, const float* __restrict__ coef, float eps, int n, int np,
                 T* __restrict__ out, long long ldo) {
  __shared__ float red[96];
  const long long row = blockIdx.x;
  const TZ* src = z + row * ldz;
  pdl_wait();
  pdl_trigger();
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

template <typename T, typename TY>
static cudaError_t launch_layer_norm(const long long* ids, const TY* y, long long ldy, int vocab, const float* wy, float* x, const float* w,
                                     float eps, int rows, int n, int np, T* h, cudaStream_t s) {
  auto go = [&](auto k, int threads) { return launch_pdl(k, dim3(rows), dim3(threads), 0, s, ids, y, ldy, vocab, wy, x, w, eps, n, np, h); };
  if (np <= 1024) return go(layer_norm_residual_kernel<T, TY, 128, 1>, 128);
  if (np <= 2048) return go(layer_norm_residual_kernel<T, TY, 128, 2>, 128);
  if (np <= 4096) return go(layer_norm_residual_kernel<T, TY, 256, 2>, 256);
  return go(layer_norm_residual_kernel<T, TY, 256, 4>, 256);
}

cudaError_t layer_norm_residual(bool f32, bool y_f32, const long long* ids, const void* y, long long ldy, int vocab, const float* wy, float* x,
                                const float* w, float eps, int rows, int n, int np, void* h, cudaStream_t s) {
  if (rows <= 0 || n <= 0 || n > np || np > 8192 || (np & 7) || (ldy & 7) || ldy < np || (ids && vocab <= 0) || (f32 && !y_f32))
    return cudaErrorInvalidValue;
  if (f32) return launch_layer_norm(ids, (const float*)y, ldy, vocab, wy, x, w, eps, rows, n, np, (float*)h, s);
  if (y_f32) return launch_layer_norm(ids, (const float*)y, ldy, vocab, wy, x, w, eps, rows, n, np, (bf16*)h, s);
  return launch_layer_norm(ids, (const bf16*)y, ldy, vocab, wy, x, w, eps, rows, n, np, (bf16*)h, s);
}

cudaError_t poly_norm(bool f32, bool z_f32, const void* z, long long ldz, const float* coef, float eps, int rows, int n, int np,
                      void* out, long long ldo, cudaStream_t s) {
  if (rows <= 0 || n <= 0 || n > np || (np & 7) || (ldz & 7) || (ldo & 7)) return cudaErrorInvalidValue;
  if (f32 && !z_f32) return cudaErrorInvalidValue;
  if (f32) return launch_pdl(poly_norm_kernel<float, float>, dim3(rows), dim3(256), 0, s, (const float*)z, ldz, coef, eps, n, np, (float*)out, ldo);
  if (z_f32) return launch_pdl(poly_norm_kernel<bf16, float>, dim3(rows), dim3(256), 0, s, (const float*)z, ldz, coef, eps, n, np, (bf16*)out, ldo);
  return launch_pdl(poly_norm_kernel<bf16, bf16>, dim3(rows), dim3(256), 0, s, (const bf16*)z, ldz, coef, eps, n, np, (bf16*)out, ldo);
}

}  // namespace serve
}  // namespace nc
