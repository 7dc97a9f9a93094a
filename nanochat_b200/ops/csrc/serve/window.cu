// Window attention over a paged store whose keys, unrotated, are also the values.
//
//   window_post       queries rotated in place, the rows' entries [rotated keys | keys] into the store (and a dense copy)
//   window_attention  any size and type: a CTA per (head, row), plain dots over the stored entries of the window
// Prompts in bf16 run on the tensor-core kernel of attention.cu from the dense copy, a step's rows on step.cu.
#include "common.cuh"

namespace nc {
namespace serve {

namespace {

// v[0 .. 8) of a head from entry i0 on: pairs (2i, 2i + 1) below `dims` turn by cs[i] = (cos, sin)
__device__ __forceinline__ void rotate8(float (&v)[8], int i0, int dims, const float2* cs) {
#pragma unroll
  for (int j = 0; j < 8; j += 2) {
    if (i0 + j < dims) {
      const float2 t = cs[(i0 + j) >> 1];
      const float a = v[j], b = v[j + 1];
      v[j] = a * t.x - b * t.y;
      v[j + 1] = b * t.x + a * t.y;
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128)
window_post_kernel(const WindowAttn d, T* dense, long long ldd, int* status) {
  extern __shared__ float2 s_cs[];
  const int row = blockIdx.x;
  int seq;
  const int pos = row_position(d.pos, row, seq);
  for (int i = threadIdx.x; i < d.dims / 2; i += blockDim.x) s_cs[i] = turn_of(pos, d.freq, i, d.dims / 2);
  const long long off = token_offset(d.pg, seq, pos);
  if (off < 0 && threadIdx.x == 0 && status) atomicCAS(status, 0, (ST_BAD_ARG << 24) | 0x57044);   // no page: not stored
  __syncthreads();
  T* z = const_cast<T*>((const T*)d.z) + row * d.ldz;
  T* entry = off < 0 ? nullptr : (T*)d.pg.pool + off;
  T* copy = dense ? dense + row * ldd : nullptr;
  const int nq = d.heads * d.dp, nk = d.kv_heads * d.dp;
  for (int c = threadIdx.x * 8; c < nq + nk; c += blockDim.x * 8) {
    float v[8];
    if (c < nq) {
      load8(z + d.q_off + c, v);
      rotate8(v, c % d.dp, d.dims, s_cs);
      store8(z + d.q_off + c, v);
    } else {
      const int k = c - nq;
      load8(z + d.k_off + k, v);
      if (entry) store8(entry + nk + k, v);
      if (copy) store8(copy + nk + k, v);
      rotate8(v, k % d.dp, d.dims, s_cs);
      if (entry) store8(entry + k, v);
      if (copy) store8(copy + k, v);
    }
  }
}

// grid (rows, heads), 128 threads; dynamic shared memory: 2 dp floats
template <typename T>
__global__ void __launch_bounds__(128)
window_attention_kernel(const WindowAttn d) {
  extern __shared__ float sm[];
  __shared__ float s_p[128];
  __shared__ long long s_off[128];
  __shared__ float s_red[8];
  const int h = blockIdx.y, row = blockIdx.x, kvh = h / (d.heads / d.kv_heads);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int k_at = kvh * d.dp, v_at = (d.kv_heads + kvh) * d.dp;
  float* sq = sm;
  float* so = sm + d.dp;
  int seq;
  const int pos = row_position(d.pos, row, seq);
  const int begin = d.window > 0 ? max(0, pos - d.window + 1) : 0;
  const T* q = (const T*)d.z + row * d.ldz + d.q_off + (long long)h * d.dp;
  for (int c = tid; c < d.dp; c += 128) { sq[c] = to_f(q[c]); so[c] = 0.f; }
  float M = NEG_BIG, L = 0.f;
  for (int tile = begin; tile <= pos; tile += 128) {
    __syncthreads();
    const int j = tile + tid;
    float s = NEG_BIG;
    long long off = -1;
    if (j <= pos) {
      off = token_offset(d.pg, seq, j);
      if (off >= 0) {
        const T* e = (const T*)d.pg.pool + off + k_at;
        float a = 0.f;
        for (int c = 0; c < d.dp; c += 8) {
          float f[8];
          load8(e + c, f);
#pragma unroll
          for (int i = 0; i < 8; ++i) a += f[i] * sq[c + i];
        }
        s = a * d.scale;
        if (d.softcap > 0.f) s = d.softcap * tanhf(s / d.softcap);
      }
    }
    s_off[tid] = off;
    const float mx = warp_max(s);
    if (lane == 0) s_red[warp] = mx;
    __syncthreads();
    const float m_new = fmaxf(M, fmaxf(fmaxf(s_red[0], s_red[1]), fmaxf(s_red[2], s_red[3])));
    const float p = off >= 0 ? expf(s - m_new) : 0.f;
    s_p[tid] = p;
    const float ps = warp_sum(p);
    if (lane == 0) s_red[4 + warp] = ps;
    __syncthreads();
    const float alpha = expf(M - m_new);
    L = L * alpha + (s_red[4] + s_red[5]) + (s_red[6] + s_red[7]);
    const int cnt = min(128, pos + 1 - tile);
    for (int c = tid; c < d.dp; c += 128) {
      float o = so[c] * alpha;
      for (int k = 0; k < cnt; ++k)
        if (s_off[k] >= 0) o += s_p[k] * to_f(((const T*)d.pg.pool)[s_off[k] + v_at + c]);
      so[c] = o;
    }
    M = m_new;
  }
  const float f = L > 0.f ? d.out_scale / L : 0.f;
  T* y = (T*)d.y + row * d.ldy + (long long)h * d.dp;
  for (int c = tid; c < d.dp; c += 128) y[c] = from_f<T>(so[c] * f);
}

bool window_ok(const WindowAttn& d) {
  const Pages& p = d.pg;
  return d.rows > 0 && d.heads > 0 && d.heads <= 65535 && d.kv_heads > 0 && d.heads % d.kv_heads == 0 && d.dp > 0 && !(d.dp & 7) &&
         d.dp <= 2048 && d.dims >= 0 && d.dims <= d.dp && !(d.dims & 1) && !(d.ldz & 7) && !(d.q_off & 7) && !(d.k_off & 7) && p.pool && p.table &&
         p.max_pages > 0 && p.shift >= 0 && p.shift <= 16 && p.n_pages > 0 && p.width == 2 * d.kv_heads * d.dp && d.pos.lens && d.pos.per_seq > 0;
}

}  // namespace

cudaError_t window_post(const WindowAttn& d, void* dense, long long ldd, int* status, cudaStream_t s) {
  if (!window_ok(d) || (dense && ((ldd & 7) || ldd < d.pg.width)) || d.f32 != d.z_f32) return cudaErrorInvalidValue;
  const size_t smem = sizeof(float2) * (d.dims / 2 + 1);
  if (d.f32) window_post_kernel<float><<<d.rows, 128, smem, s>>>(d, (float*)dense, ldd, status);
  else window_post_kernel<bf16><<<d.rows, 128, smem, s>>>(d, (bf16*)dense, ldd, status);
  return cudaGetLastError();
}

cudaError_t window_attention(const WindowAttn& d, cudaStream_t s) {
  if (!window_ok(d) || d.y == nullptr || d.f32 != d.z_f32) return cudaErrorInvalidValue;
  const dim3 grid(d.rows, d.heads);
  const size_t smem = 2 * d.dp * sizeof(float);
  if (d.f32) window_attention_kernel<float><<<grid, 128, smem, s>>>(d);
  else window_attention_kernel<bf16><<<grid, 128, smem, s>>>(d);
  return cudaGetLastError();
}

}  // namespace serve
}  // namespace nc
