// One row's entry of the latent store, written by one block: [ norm(z[0:kv_rank]) * w, zeros | rotated key part, zeros ].
#pragma once

#include "common.cuh"

namespace nc {
namespace serve {

// zc: the row's latent before its norm; zr: its key part before rotation. dst / dense: the store's entry and an
// optional dense copy (either may be null). All threads of the block take part. `red`: 32 floats.
template <typename T, typename TZ>
__device__ __forceinline__ void store_latent(const TZ* zc, const TZ* zr, int kv_rank, int kvp, const float* kv_w, float eps,
                                             int rot_dim, int rp, int dims, const float* freq, int position, T* dst,
                                             T* dense, float* red) {
  float ss[1] = {0.f};
  for (int c = threadIdx.x; c < kv_rank; c += blockDim.x) { const float v = to_f(zc[c]); ss[0] += v * v; }
  block_sum<1>(ss, red);
  const float r = inv_rms(ss[0], kv_rank, eps);
  for (int c = threadIdx.x; c < kvp; c += blockDim.x) {
    const T v = from_f<T>(c < kv_rank ? to_f(zc[c]) * r * kv_w[c] : 0.f);
    if (dst) dst[c] = v;
    if (dense) dense[c] = v;
  }
  const int half = dims >> 1;
  for (int i = threadIdx.x; i < rp; i += blockDim.x) {
    float v = 0.f;
    if (i < dims) {
      const int p = i < half ? i : i - half;
      float sn, cs;
      sincosf((float)position * freq[p], &sn, &cs);
      const float a = to_f(zr[p]), b = to_f(zr[p + half]);
      v = i < half ? a * cs - b * sn : b * cs + a * sn;
    } else if (i < rot_dim) {
      v = to_f(zr[i]);
    }
    const T o = from_f<T>(v);
    if (dst) dst[kvp + i] = o;
    if (dense) dense[kvp + i] = o;
  }
}

}  // namespace serve
}  // namespace nc
