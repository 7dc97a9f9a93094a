// Mixture of experts.
//
// Prompts: rows are grouped by expert (every group padded to the 128-row tile of the tensor-core GEMM, whose tiles then
// belong to one expert each; see GemmDesc::m_group), and a row's chosen outputs are summed by the residual kernel.
//   route_topk -> plan_groups -> gather_groups -> grouped GEMM -> silu_mul -> grouped GEMM
// A row's place inside its group comes from an atomic counter, so it varies; its values do not depend on it.
//
// Few rows, and float: one matrix-vector product per (row, chosen expert), a CTA per four outputs with K split over its
// threads. (bf16 decode steps read each expert once for all their rows instead, see gemv.cu.)
#include "common.cuh"

namespace nc {
namespace serve {

namespace {

__global__ void __launch_bounds__(128)
route_topk_kernel(const float* __restrict__ logits, long long ld, int rows, int experts, int top, int* __restrict__ idx,
                  float* __restrict__ wt, int* __restrict__ counts, int* __restrict__ rank) {
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  pdl_wait();
  pdl_trigger();
  const float* z = logits + row * ld;
  float v = INFINITY, best = 0.f, sum = 0.f;
  int i = -1;
  for (int k = 0; k < top; ++k) {
    float nv; int ni;
    next_best(z, experts, v, i, lane, nv, ni);
    v = nv; i = ni;
    if (k == 0) best = v;
    const float e = expf(v - best);
    sum += e;
    if (lane == 0) {
      idx[(long long)row * top + k] = i;
      wt[(long long)row * top + k] = e;
      if (counts) rank[(long long)row * top + k] = atomicAdd(counts + i, 1);
    }
  }
  __syncwarp();
  const float inv = 1.f / sum;
  if (lane == 0)
    for (int k = 0; k < top; ++k) wt[(long long)row * top + k] *= inv;
}

// one block: exclusive sum of the groups' padded sizes, then the tiles' groups
__global__ void __launch_bounds__(256)
plan_groups_kernel(const int* __restrict__ counts, int experts, int* __restrict__ offsets, int* __restrict__ tile_group, int tiles) {
  __shared__ int s_used;
  if (threadIdx.x < 32) {
    int base = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int padded = e < experts ? (counts[e] + 127) / 128 * 128 : 0;
      int incl = padded;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int t = __shfl_up_sync(0xffffffffu, incl, o);
        if ((int)threadIdx.x >= o) incl += t;
      }
      if (e < experts) {
        const int first = base + incl - padded;
        offsets[e] = first;
        for (int t = first / 128; t < (first + padded) / 128 && t < tiles; ++t) tile_group[t] = e;
      }
      base += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (threadIdx.x == 0) s_used = base / 128;
  }
  __syncthreads();
  for (int t = s_used + threadIdx.x; t < tiles; t += blockDim.x) tile_group[t] = -1;
}

__global__ void __launch_bounds__(128)
gather_groups_kernel(const bf16* __restrict__ h, long long ldh, int top, int np, const int* __restrict__ idx,
                     const int* __restrict__ rank, const int* __restrict__ offsets, int* __restrict__ slot, bf16* __restrict__ xg) {
  const long long i = blockIdx.x;
  const long long to = offsets[idx[i]] + rank[i];
  if (threadIdx.x == 0) slot[i] = (int)to;
  const uint4* src = reinterpret_cast<const uint4*>(h + i / top * ldh);
  uint4* dst = reinterpret_cast<uint4*>(xg + to * np);
  for (int c = threadIdx.x; c < np / 8; c += 128) dst[c] = src[c];
}

__global__ void __launch_bounds__(256)
silu_mul_kernel(const bf16* __restrict__ gu, int fp, const int* __restrict__ tile_group, bf16* __restrict__ act) {
  const long long row = blockIdx.x;
  if (tile_group[row / 128] < 0) return;
  for (int c = threadIdx.x * 8; c < fp; c += 2048) {
    float g[8], u[8];
    load8(gu + row * 2 * fp + c, g);
    load8(gu + row * 2 * fp + fp + c, u);
#pragma unroll
    for (int j = 0; j < 8; ++j) g[j] = g[j] * fast_sigmoidf(g[j]) * u[j];
    store8(act + row * fp + c, g);
  }
}

constexpr int COLS = 4;

// Sums COLS values per thread over the block; thread c < COLS gets value c.
__device__ __forceinline__ float block_cols(float (&v)[COLS], float (*smem)[COLS]) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float t = warp_sum_many<COLS>(v, lane);
  if ((lane & 7) == 0) smem[warp][lane >> 3] = t;
  __syncthreads();
  float r = 0.f;
  if (threadIdx.x < COLS) {
#pragma unroll
    for (int w = 0; w < 8; ++w) r += smem[w][threadIdx.x];
  }
  return r;
}

// grid (rows * top, ceil(fp / 4))
template <typename T>
__global__ void __launch_bounds__(256)
expert_gate_up_kernel(const T* __restrict__ h, long long ldh, int K, const T* __restrict__ Wgu, int fp, Routing rt,
                      T* __restrict__ act) {
  __shared__ float s_g[8][COLS], s_u[8][COLS];
  const int row = blockIdx.x / rt.top, k = blockIdx.x - row * rt.top, n0 = blockIdx.y * COLS;
  pdl_wait();
  pdl_trigger();
  const long long e = rt.idx[(long long)row * rt.top + k];
  const T* wg = Wgu + e * 2 * fp * K;
  const T* wu = wg + (long long)fp * K;
  float g[COLS] = {0.f, 0.f, 0.f, 0.f}, u[COLS] = {0.f, 0.f, 0.f, 0.f};
  for (int c = threadIdx.x * 8; c < K; c += 2048) {
    Raw8<T> rg[COLS], ru[COLS];
#pragma unroll
    for (int r = 0; r < COLS; ++r) {
      const long long n = min(n0 + r, fp - 1);
      rg[r] = raw8(wg + n * K + c);
      ru[r] = raw8(wu + n * K + c);
    }
    float x[8], f[8];
    load8(h + row * ldh + c, x);
#pragma unroll
    for (int r = 0; r < COLS; ++r) {
      unraw8(rg[r], f);
#pragma unroll
      for (int j = 0; j < 8; ++j) g[r] += f[j] * x[j];
      unraw8(ru[r], f);
#pragma unroll
      for (int j = 0; j < 8; ++j) u[r] += f[j] * x[j];
    }
  }
  const float gs = block_cols(g, s_g), us = block_cols(u, s_u);
  if (threadIdx.x < COLS && n0 + (int)threadIdx.x < fp)
    act[(long long)blockIdx.x * fp + n0 + threadIdx.x] = from_f<T>(gs * sigmoidf(gs) * us);
}

// grid (rows, ceil(N / 4))
template <typename T>
__global__ void __launch_bounds__(256)
expert_down_kernel(const ExpertDown d) {
  __shared__ float s_acc[8][COLS];
  const int row = blockIdx.x, n0 = blockIdx.y * COLS, top = d.rt.top;
  pdl_wait();
  pdl_trigger();
  float acc[COLS] = {0.f, 0.f, 0.f, 0.f};
  for (int t = 0; t < top; ++t) {
    const T* w = (const T*)d.Wdown + (long long)d.rt.idx[(long long)row * top + t] * d.N * d.fp;
    const T* a = (const T*)d.act + ((long long)row * top + t) * d.fp;
    const float wt = d.rt.wt[(long long)row * top + t];
    for (int c = threadIdx.x * 8; c < d.fp; c += 2048) {
      Raw8<T> rw[COLS];
#pragma unroll
      for (int r = 0; r < COLS; ++r) rw[r] = raw8(w + (long long)min(n0 + r, d.N - 1) * d.fp + c);
      float x[8], f[8];
      load8(a + c, x);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] *= wt;
#pragma unroll
      for (int r = 0; r < COLS; ++r) {
        unraw8(rw[r], f);
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[r] += f[j] * x[j];
      }
    }
  }
  const float v = block_cols(acc, s_acc);
  const int n = n0 + threadIdx.x;
  if (threadIdx.x < COLS && n < d.N) ((T*)d.y)[row * d.ldy + n] = from_f<T>(v);
}

bool routing_ok(const Routing& r) {
  return r.experts > 0 && r.top > 0 && r.top <= r.experts && r.idx != nullptr && r.wt != nullptr;
}

}  // namespace

cudaError_t route_topk(const float* logits, long long ld, int rows, int experts, int top, int* idx, float* wt,
                       int* counts, int* rank, cudaStream_t s) {
  if (rows <= 0 || experts <= 0 || top <= 0 || top > experts || ld < experts || (counts != nullptr) != (rank != nullptr))
    return cudaErrorInvalidValue;
  return launch_pdl(route_topk_kernel, dim3((rows + 3) / 4), dim3(128), 0, s, logits, ld, rows, experts, top, idx, wt, counts, rank);
}

cudaError_t plan_groups(const int* counts, int experts, int* offsets, int* tile_group, int tiles, cudaStream_t s) {
  if (experts <= 0 || tiles <= 0) return cudaErrorInvalidValue;
  plan_groups_kernel<<<1, 256, 0, s>>>(counts, experts, offsets, tile_group, tiles);
  return cudaGetLastError();
}

cudaError_t gather_groups(const void* h, long long ldh, int rows, int top, int np, const int* idx, const int* rank,
                          const int* offsets, int* slot, void* xg, cudaStream_t s) {
  if (rows <= 0 || top <= 0 || np <= 0 || (np & 7) || (ldh & 7)) return cudaErrorInvalidValue;
  gather_groups_kernel<<<rows * top, 128, 0, s>>>((const bf16*)h, ldh, top, np, idx, rank, offsets, slot, (bf16*)xg);
  return cudaGetLastError();
}

cudaError_t silu_mul(const void* gu, int rows, int fp, const int* tile_group, void* act, cudaStream_t s) {
  if (rows <= 0 || fp <= 0 || (fp & 7)) return cudaErrorInvalidValue;
  silu_mul_kernel<<<rows, 256, 0, s>>>((const bf16*)gu, fp, tile_group, (bf16*)act);
  return cudaGetLastError();
}

cudaError_t expert_gate_up(bool f32, const void* h, long long ldh, int rows, int K, const void* Wgu, int fp,
                           const Routing& rt, void* act, cudaStream_t s) {
  if (rows <= 0 || K <= 0 || (K & 7) || (ldh & 7) || fp <= 0 || (fp & 7) || fp / COLS > 65535 || !routing_ok(rt)) return cudaErrorInvalidValue;
  const dim3 grid(rows * rt.top, (fp + COLS - 1) / COLS);
  if (f32) return launch(true, expert_gate_up_kernel<float>, grid, dim3(256), 0, s, (const float*)h, ldh, K, (const float*)Wgu, fp, rt, (float*)act);
  return launch(true, expert_gate_up_kernel<bf16>, grid, dim3(256), 0, s, (const bf16*)h, ldh, K, (const bf16*)Wgu, fp, rt, (bf16*)act);
}

cudaError_t expert_down(const ExpertDown& d, cudaStream_t s) {
  if (d.rows <= 0 || d.fp <= 0 || (d.fp & 7) || d.N <= 0 || d.N / COLS > 65534 || !routing_ok(d.rt) || !d.y)
    return cudaErrorInvalidValue;
  const dim3 grid(d.rows, (d.N + COLS - 1) / COLS);
  if (d.f32) return launch(true, expert_down_kernel<float>, grid, dim3(256), 0, s, d);
  return launch(true, expert_down_kernel<bf16>, grid, dim3(256), 0, s, d);
}

}  // namespace serve
}  // namespace nc
