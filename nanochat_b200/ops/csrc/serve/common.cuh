// Building blocks of the serving kernels: 8-wide typed loads and stores, block reductions, the paged store address,
// expert selection, and the launch helper for chains of short kernels (programmatic dependent launch).
// A row always has a multiple of 8 elements; entries past a row's real size are zero.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../host_utils.cuh"
#include "../ptx.cuh"
#include "serve.h"

namespace nc {
namespace serve {

using bf16 = __nv_bfloat16;

// ------------------------------------------------------------------ typed vectors of 8
__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
  const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y), c = unpack_bf16(u.z), d = unpack_bf16(u.w);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
}
__device__ __forceinline__ void load8(const bf16* p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void store8(bf16* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }

// Weight rows are read once per step: keep them out of L1. Raw form, so that the request can be issued before the
// wait on the preceding kernel.
template <typename T> struct Raw8;
template <> struct Raw8<bf16> { uint4 a; };
template <> struct Raw8<float> { uint4 a, b; };
__device__ __forceinline__ uint4 ld_once(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
__device__ __forceinline__ Raw8<bf16> raw8(const bf16* p) { return {ld_once(p)}; }
__device__ __forceinline__ Raw8<float> raw8(const float* p) { return {ld_once(p), ld_once(p + 4)}; }
__device__ __forceinline__ void unraw8(const Raw8<bf16>& r, float (&f)[8]) { unpack8(r.a, f); }
__device__ __forceinline__ void unraw8(const Raw8<float>& r, float (&f)[8]) {
  f[0] = __uint_as_float(r.a.x); f[1] = __uint_as_float(r.a.y); f[2] = __uint_as_float(r.a.z); f[3] = __uint_as_float(r.a.w);
  f[4] = __uint_as_float(r.b.x); f[5] = __uint_as_float(r.b.y); f[6] = __uint_as_float(r.b.z); f[7] = __uint_as_float(r.b.w);
}

// ------------------------------------------------------------------------- reductions
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Sums of N values over the block, returned to every thread. `smem` holds N * 32 floats; the leading barrier makes
// it reusable by back-to-back calls.
template <int N>
__device__ __forceinline__ void block_sum(float (&v)[N], float* smem) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(v[i]);
  __syncthreads();
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) smem[i * 32 + warp] = v[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(lane < warps ? smem[i * 32 + lane] : 0.f);
}

__host__ __device__ constexpr int pow2_ceil(int n) { int p = 1; while (p < n) p <<= 1; return p; }
__host__ __device__ constexpr int ilog2(int n) { int l = 0; while ((1 << l) < n) ++l; return l; }

// Warp-wide sums of NV values per lane (NV a power of two <= 32) with a halving exchange: lane l ends up with the sum
// of value l >> (5 - log2 NV).
template <int NV>
__device__ __forceinline__ float warp_sum_many(float (&v)[NV], int lane) {
  constexpr int LOG = ilog2(NV);
#pragma unroll
  for (int s = 0; s < LOG; ++s) {
    const int off = 16 >> s, half = NV >> (s + 1);
    const bool upper = (lane & off) != 0;
#pragma unroll
    for (int i = 0; i < half; ++i) {
      const float send = upper ? v[i] : v[i + half];
      const float keep = upper ? v[i + half] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
    }
  }
  float r = v[0];
#pragma unroll
  for (int off = 16 >> LOG; off >= 1; off >>= 1) r += __shfl_xor_sync(0xffffffffu, r, off);
  return r;
}

// -------------------------------------------------------------------------- small math
__device__ __forceinline__ float sigmoidf(float v) { return 1.f / (1.f + expf(-v)); }
// next to bf16 values: a few units in the last place of a float do not matter
__device__ __forceinline__ float fast_sigmoidf(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }
template <typename T> __device__ __forceinline__ float sigmoid_of(float v) { return sizeof(T) == 4 ? sigmoidf(v) : fast_sigmoidf(v); }
__device__ __forceinline__ float inv_rms(float sumsq, int n, float eps) { return 1.f / sqrtf(sumsq / n + eps); }

// ------------------------------------------------------------------------- paged store
// Offset (in elements) of token t of sequence s, or -1 when the table has no room for it.
__device__ __forceinline__ long long token_offset(const Pages& pg, int s, int t) {
  const int p = t >> pg.shift;
  if (t < 0 || p >= pg.max_pages) return -1;
  const int page = pg.table[(long long)s * pg.max_pages + p];
  if (page < 0 || page >= pg.n_pages) return -1;
  return ((long long)page << pg.shift | (t & ((1 << pg.shift) - 1))) * pg.width;
}

// (cos, sin) of position * f, f = freq[i] + freq[half + i] (a frequency and what its float leaves over): the product's own
// rounding error and the left-over enter to first order, so the angle is good to 2^-24 of a turn's size at any position
__device__ __forceinline__ float2 turn_of(int position, const float* freq, int i, int half) {
  const float p = (float)position, f = freq[i], a = p * f;
  const float rest = fmaf(p, f, -a) + p * freq[half + i];
  float sn, cs;
  sincosf(a, &sn, &cs);
  return make_float2(cs - rest * sn, sn + rest * cs);
}

// ------------------------------------------------------------------- rows, key ranges
constexpr float NEG_BIG = -1.0e30f;
__device__ __forceinline__ int row_position(const RowPos& p, int row, int& seq) {
  seq = row / p.per_seq;
  return p.lens[seq] + row - seq * p.per_seq;
}

struct KeyRange { int begin, end; };       // this split's keys
__device__ __forceinline__ KeyRange split_keys(int pos, int window, int splits, int split, int tile) {
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int n = pos - lo + 1;
  int chunk = (n + splits - 1) / splits;
  chunk = (chunk + tile - 1) / tile * tile;
  KeyRange r;
  r.begin = lo + split * chunk;
  r.end = min(pos + 1, r.begin + chunk);
  return r;
}

// ---------------------------------------------------------------------------- routing
// One warp: the entry that follows (last_v, last_i) in the order of falling value, rising index among equals.
__device__ __forceinline__ void next_best(const float* z, int n, float last_v, int last_i, int lane, float& v, int& i) {
  v = -INFINITY; i = 0x7fffffff;
  for (int e = lane; e < n; e += 32) {
    const float t = z[e];
    const bool after = t < last_v || (t == last_v && e > last_i);
    if (after && (t > v || (t == v && e < i))) { v = t; i = e; }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
  }
  if (i < 0 || i >= n) i = 0;          // no ordered entry left (logits that are not numbers): stay in bounds
}

// ------------------------------------------------- programmatic dependent launch chains
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

template <typename... KArgs, typename... Args>
cudaError_t launch_pdl(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = s;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  at[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = at; cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kern, static_cast<KArgs>(args)...);
}

// plain launch, or one that may overlap the end of the kernel before it
template <typename... KArgs, typename... Args>
cudaError_t launch(bool pdl, void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args... args) {
  if (pdl) return launch_pdl(kern, grid, block, smem, s, args...);
  kern<<<grid, block, smem, s>>>(static_cast<KArgs>(args)...);
  return cudaGetLastError();
}

// This CTA's slice of the weights a later kernel will stream, requested into L2.
__device__ __forceinline__ void prefetch_l2_slice(const NextWeights& next, long long cta, long long ctas) {
  if (next.ptr == nullptr || threadIdx.x != 0) return;
  long long chunk = ((next.bytes + ctas - 1) / ctas + 15) & ~15ll;
  const long long begin = cta * chunk;
  if (begin >= next.bytes) return;
  long long n = next.bytes - begin < chunk ? next.bytes - begin : chunk;
  n &= ~15ll;
  if (n <= 0) return;
  asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"((const char*)next.ptr + begin), "r"((uint32_t)n) : "memory");
}

}  // namespace serve
}  // namespace nc
