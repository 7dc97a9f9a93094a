// Recurrences over a per-sequence state (dp x vp floats a head): the gated delta rule and linear attention with a fixed
// decay per head, for portions of several tokens.
//
//   delta_prepare     short convolution + silu of queries, keys and values, inverse norms, step sizes, log decays
//   silu_rows         the activation of the fixed-decay inputs
//   recurrence_scan   token by token, the state in registers: float, short portions, wide heads
//   recurrence_chunks chunks of 64 tokens, two kernels:
//       gram   (parallel over chunks) A = (Q K^T) with decays, causal; for the delta rule also the inverse of the unit
//              triangular system that the tokens of a chunk solve, T = (1 + strict(beta K K^T with decays))^-1 beta
//       scan   (sequential over chunks, one CTA per 16 state columns)
//                 R = V - decayed K S,  U = T R        delta rule;   U = V  fixed decay
//                 O = decayed Q S + A U
//                 S = decayed S + K^T (decayed U)
//   norm_gate         RMS norm and gate of what a recurrence read out, and the convolution's last inputs
//
// Exactness: the products run on bf16 operands, so every operand that is a float (the state, T, A, U, R) enters as the sum
// of two bf16 values, and what scales rows (inverse norms, decays) is applied to accumulators, not to operands: keys,
// queries and values are the bf16 activations themselves. The state is float from chunk to chunk.
#include "mma.cuh"

namespace nc {
namespace serve {

namespace {

template <typename T> __device__ __forceinline__ float silu_of(float v) { return v * sigmoid_of<T>(v); }

__device__ __forceinline__ void load4(const float* p, float (&f)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
}
__device__ __forceinline__ void load4(const bf16* p, float (&f)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
__device__ __forceinline__ void store4(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
__device__ __forceinline__ void store4(bf16* p, const float (&f)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]));
}

// ---------------------------------------------------------------------------- prepare
constexpr int PREP_TOKENS = 8;         // tokens a warp walks through

// grid (token groups of a sequence, ceil(jobs / 4), sequences), a warp per job: query heads, key heads, value heads.
// TAPS > 0: at most TAPS taps, the inputs slide through registers; 0: any number, re-read
template <typename T, typename TZ, int TAPS>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const DeltaInputs d, T* __restrict__ act, float* __restrict__ norms, float* __restrict__ beta_g) {
  const int lane = threadIdx.x & 31, job = blockIdx.y * 4 + (threadIdx.x >> 5);
  const int G = d.kv_heads, H = d.heads, per_seq = d.pos.per_seq, seq = blockIdx.z;
  if (job >= 2 * G + H) return;
  const int t0 = blockIdx.x * PREP_TOKENS, n = min(PREP_TOKENS, per_seq - t0);
  const int channels = 2 * G * d.dp + H * d.vp, size = job < 2 * G ? d.dp : d.vp;
  const int ch0 = job < 2 * G ? job * d.dp : 2 * G * d.dp + (job - 2 * G) * d.vp;
  const int start = d.pos.lens[seq];
  const long long row0 = (long long)seq * per_seq;
  const float* ring = d.ring.ptr + seq * d.ring.seq_stride;
  auto fetch = [&](int t, int ch, float (&x)[4]) {
    if (t >= 0) {
      load4((const TZ*)d.z + (row0 + t) * d.ldz + ch, x);
    } else if (start + t >= 0) {
      load4(ring + (long long)((start + t) % d.taps) * channels + ch, x);
    } else {
      x[0] = x[1] = x[2] = x[3] = 0.f;
    }
  };
  float ss[PREP_TOKENS];
#pragma unroll
  for (int t = 0; t < PREP_TOKENS; ++t) ss[t] = 0.f;
  for (int c = lane * 4; c < size; c += 128) {
    const int ch = ch0 + c;
    constexpr int HELD = TAPS > 0 ? TAPS : 1;
    float w[HELD][4], x[HELD][4];                       // tap i meets the token i places back
    if (TAPS > 0) {
#pragma unroll
      for (int i = 0; i < HELD; ++i) {
        if (i < d.taps) {
          load4(d.conv + (long long)(d.taps - 1 - i) * channels + ch, w[i]);
          if (i > 0) fetch(t0 - i, ch, x[i]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j) w[i][j] = x[i][j] = 0.f;
        }
      }
    }
#pragma unroll
    for (int t = 0; t < PREP_TOKENS; ++t) {
      if (t >= n) break;
      float a[4] = {0.f, 0.f, 0.f, 0.f};
      if (TAPS > 0) {
        fetch(t0 + t, ch, x[0]);
#pragma unroll
        for (int i = 0; i < HELD; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) a[j] += w[i][j] * x[i][j];
#pragma unroll
        for (int i = HELD - 1; i > 0; --i)
#pragma unroll
          for (int j = 0; j < 4; ++j) x[i][j] = i < d.taps ? x[i - 1][j] : 0.f;
      } else {
        for (int i = 0; i < d.taps; ++i) {
          load4(d.conv + (long long)(d.taps - 1 - i) * channels + ch, w[0]);
          fetch(t0 + t - i, ch, x[0]);
#pragma unroll
          for (int j = 0; j < 4; ++j) a[j] += w[0][j] * x[0][j];
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        a[j] = to_f(from_f<T>(silu_of<T>(a[j])));       // the norm is that of the vector that is stored
        ss[t] += a[j] * a[j];
      }
      store4(act + (row0 + t0 + t) * channels + ch, a);
    }
  }
  if (job < 2 * G) {
#pragma unroll
    for (int t = 0; t < PREP_TOKENS; ++t) {
      const float r = 1.f / sqrtf(warp_sum(ss[t]) + 1e-6f);
      if (lane == 0 && t < n) norms[(row0 + t0 + t) * 2 * G + job] = job < G ? r / sqrtf((float)d.dim) : r;
    }
  } else if (lane < n) {
    const int h = job - 2 * G;
    const float* in = d.ba + (row0 + t0 + lane) * d.ldba;
    const float a = in[d.a_off + h] + d.dt_bias[h];
    float* out = beta_g + (row0 + t0 + lane) * 2 * H;
    out[h] = sigmoidf(in[h]);
    out[H + h] = d.neg_a[h] * (a > 20.f ? a : log1pf(expf(a)));
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
silu_rows_kernel(const T* __restrict__ z, long long ldz, int rows, int n, T* __restrict__ act, long long lda) {
  const int per = n / 8;
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x, row = i / per;
  if (row >= rows) return;
  const int c = (int)(i - row * per) * 8;
  float v[8];
  load8(z + row * ldz + c, v);
#pragma unroll
  for (int j = 0; j < 8; ++j) v[j] = silu_of<T>(v[j]);
  store8(act + row * lda + c, v);
}

// ------------------------------------------------------------------------------- scan
// grid (ceil(vp / 16), heads, sequences), 4 warps of 4 state columns, lane l holds rows l, l + 32, ...
template <typename T, bool DELTA, int DPL>
__global__ void __launch_bounds__(128)
recurrence_scan_kernel(const Recurrence r) {
  const int lane = threadIdx.x & 31, h = blockIdx.y, seq = blockIdx.z, kvh = h / (r.heads / r.kv_heads);
  const int v0 = blockIdx.x * 16 + (threadIdx.x >> 5) * 4;
  if (v0 >= r.vp) return;
  const int n = r.pos.per_seq;
  const long long row0 = (long long)seq * n;
  float* st = r.state.ptr + seq * r.state.seq_stride + (long long)h * r.dp * r.vp + v0;
  const bool fresh = r.pos.lens[seq] == 0;
  float S[DPL][4];
#pragma unroll
  for (int i = 0; i < DPL; ++i) {
    const int dd = lane + i * 32;
    if (dd < r.dp && !fresh) {
      load4(st + (long long)dd * r.vp, S[i]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) S[i][j] = 0.f;
    }
  }
  const T* base = (const T*)r.act + row0 * r.lda;
  const T* qp = base + r.q_off + kvh * r.dp;
  const T* kp = base + r.k_off + kvh * r.dp;
  const T* vp = base + r.v_off + h * r.vp + v0;
  const float g_fixed = DELTA ? 0.f : expf(r.log_decay[h]);
  float qn[DPL], kn[DPL], vn[4], sc[4];                      // the next token's inputs; sc: 1/|q|, 1/|k|, beta, log g
  auto request = [&](int t) {
#pragma unroll
    for (int i = 0; i < DPL; ++i) {
      const int dd = lane + i * 32;
      qn[i] = dd < r.dp ? to_f(qp[t * r.lda + dd]) : 0.f;
      kn[i] = dd < r.dp ? to_f(kp[t * r.lda + dd]) : 0.f;
    }
    load4(vp + t * r.lda, vn);
    if (DELTA) {
      const float* nr = r.norms + (row0 + t) * 2 * r.kv_heads;
      const float* bg = r.beta_g + (row0 + t) * 2 * r.heads;
      sc[0] = nr[kvh]; sc[1] = nr[r.kv_heads + kvh]; sc[2] = bg[h]; sc[3] = bg[r.heads + h];
    }
  };
  request(0);
  for (int t = 0; t < n; ++t) {
    float q[DPL], k[DPL], v[4], u[4];
    const float rq = DELTA ? sc[0] : 1.f, rk = DELTA ? sc[1] : 1.f, beta = DELTA ? sc[2] : 1.f, g = DELTA ? expf(sc[3]) : g_fixed;
#pragma unroll
    for (int i = 0; i < DPL; ++i) { q[i] = qn[i]; k[i] = kn[i]; }
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = vn[j];
    if (t + 1 < n) request(t + 1);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (DELTA) {
        float p = 0.f;
#pragma unroll
        for (int i = 0; i < DPL; ++i) p += S[i][j] * k[i];
        u[j] = rk * beta * (v[j] - g * rk * warp_sum(p));
      } else {
        u[j] = v[j];
      }
    }
    float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < DPL; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        S[i][j] = g * S[i][j] + k[i] * u[j];
        o[j] += S[i][j] * q[i];
      }
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] = rq * warp_sum(o[j]);
    if (lane == 0) store4((T*)r.o + (row0 + t) * r.ldo + (long long)h * r.vp + v0, o);
  }
#pragma unroll
  for (int i = 0; i < DPL; ++i) {
    const int dd = lane + i * 32;
    if (dd < r.dp) store4(st + (long long)dd * r.vp, S[i]);
  }
}

// ------------------------------------------------------------------------------ chunks
constexpr int CH = 64;                       // tokens per chunk
constexpr int TRI = CH * CH;                 // one 64 x 64 operand
constexpr int LT = CH + 8;                   // its pitch in shared memory
constexpr int SCALARS = 200;                 // floats per chunk and head: three vectors of 64, the chunk's total decay, padding
constexpr int VS = 16;                       // state columns per CTA
constexpr int LV = VS + 8;

__host__ __device__ constexpr int up16(int n) { return (n + 15) / 16 * 16; }
__host__ __device__ constexpr size_t chunk_bytes(bool delta) { return (size_t)(delta ? 4 : 2) * TRI * 2 + SCALARS * 4; }

// Inclusive sums of 64 entries, lane l holding entries 2l and 2l + 1. Double: a token that forgets nearly everything has a
// large logarithm, and the tokens after it need the small differences behind it.
__device__ __forceinline__ double cumulative_64(double a, double b, int lane, double& first) {
  double s = a + b;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double t = __shfl_up_sync(0xffffffffu, s, o);
    if (lane >= o) s += t;
  }
  first = s - b;
  return s;
}

// grid (chunks, heads, sequences), 128 threads. Row i of a chunk: scalars [0, 64) decayed 1/|k|, [64, 128) decayed 1/|q|,
// [128, 192) 1/|k| times the decay from the token to the chunk's end, [192] the decay over the whole chunk.
template <bool DELTA>
__global__ void __launch_bounds__(128)
chunk_gram_kernel(const Recurrence r, uint8_t* __restrict__ scratch) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float sB[CH], sRk[CH], sRq[CH];
  __shared__ double sG[CH];                                  // log decay from the chunk's start, each token's own included
  const int chunk = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, kvh = h / (r.heads / r.kv_heads);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = chunk * CH, n = min(CH, r.pos.per_seq - t0);
  const long long row0 = (long long)seq * r.pos.per_seq + t0;
  const int D = up16(r.dp), LD = D + 8;
  bf16* sK = reinterpret_cast<bf16*>(smem_raw);
  bf16* sQ = sK + CH * LD;
  float* sL = reinterpret_cast<float*>(smem_raw);            // takes the place of the tiles once they have been used
  constexpr int LL = CH + 4;
  const bf16* act = (const bf16*)r.act + row0 * r.lda;
  for (int i = tid; i < CH * (D / 8); i += 128) {
    const int row = i / (D / 8), c = (i - row * (D / 8)) * 8;
    const bool in = row < n && c < r.dp;
    const long long at = in ? row * r.lda + kvh * r.dp + c : 0;
    cp_async16_or_zero(sK + row * LD + c, act + (in ? r.k_off : 0) + at, in);
    cp_async16_or_zero(sQ + row * LD + c, act + (in ? r.q_off : 0) + at, in);
  }
  cp_async_commit();
  uint8_t* unit = scratch + ((long long)(seq * gridDim.x + chunk) * r.heads + h) * chunk_bytes(DELTA);
  bf16* gA = reinterpret_cast<bf16*>(unit);
  float* gS = reinterpret_cast<float*>(unit + (DELTA ? 4 : 2) * TRI * 2);
  if (warp == 0) {
    if (DELTA) {
      float lg[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = lane * 2 + e;
        const float* nr = r.norms + (row0 + i) * 2 * r.kv_heads;
        const float* bg = r.beta_g + (row0 + i) * 2 * r.heads;
        sRq[i] = i < n ? nr[kvh] : 0.f;
        sRk[i] = i < n ? nr[r.kv_heads + kvh] : 0.f;
        sB[i] = i < n ? bg[h] : 0.f;
        lg[e] = i < n ? bg[r.heads + h] : 0.f;
      }
      double first;
      const double second = cumulative_64(lg[0], lg[1], lane, first);
      sG[lane * 2] = first; sG[lane * 2 + 1] = second;
    } else {
      const float ld = r.log_decay[h];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = lane * 2 + e;
        sG[i] = (double)ld * (i + 1);
        sRq[i] = sRk[i] = i < n ? 1.f : 0.f;
      }
    }
    __syncwarp();
    const double last = sG[n - 1];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = lane * 2 + e;
      const float g = expf((float)sG[i]);
      gS[i] = g * sRk[i];
      gS[CH + i] = g * sRq[i];
      gS[2 * CH + i] = i < n ? sRk[i] * expf((float)(last - sG[i])) : 0.f;
    }
    if (lane == 0) gS[3 * CH] = expf((float)last);
  }
  cp_async_wait<0>();
  __syncthreads();
  float qk[8][4], kk[DELTA ? 8 : 1][4];
#pragma unroll
  for (int t = 0; t < 8; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) { qk[t][e] = 0.f; if (DELTA) kk[t][e] = 0.f; }
  for (int k = 0; k < D; k += 16) {
    uint32_t aq[4], ak[4];
    ldmatrix4(aq, sQ + (warp * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
    if (DELTA) ldmatrix4(ak, sK + (warp * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
#pragma unroll
    for (int t = 0; t < 8; t += 2) {
      if (t > 2 * warp + 1) break;
      uint32_t b[4];                                            // keys t * 8 .. t * 8 + 15, both halves of k
      ldmatrix4(b, sK + (t * 8 + (lane & 7) + (lane >> 4) * 8) * LD + k + ((lane >> 3) & 1) * 8);
      mma_16816(qk[t], aq, b[0], b[1]);
      mma_16816(qk[t + 1], aq, b[2], b[3]);
      if constexpr (DELTA) {
        mma_16816(kk[t], ak, b[0], b[1]);
        mma_16816(kk[t + 1], ak, b[2], b[3]);
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int t = 0; t < 8; ++t) {
    const int j = t * 8 + (lane & 3) * 2;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = warp * 16 + (lane >> 2) + half * 8;
      float a[2], l[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = j + e;
        const float decay = c <= i ? expf((float)(sG[i] - sG[c])) : 0.f;
        a[e] = c <= i ? sRq[i] * sRk[c] * decay * qk[t][half * 2 + e] : 0.f;
        if constexpr (DELTA) l[e] = c < i ? sB[i] * sRk[i] * sRk[c] * decay * kk[t][half * 2 + e] : 0.f;
      }
      if (t <= 2 * warp + 1) {
        bf16 hi[2], lo[2];
        split_bf16(a[0], hi[0], lo[0]);
        split_bf16(a[1], hi[1], lo[1]);
        *reinterpret_cast<__nv_bfloat162*>(gA + i * CH + j) = __nv_bfloat162(hi[0], hi[1]);
        *reinterpret_cast<__nv_bfloat162*>(gA + TRI + i * CH + j) = __nv_bfloat162(lo[0], lo[1]);
      }
      if constexpr (DELTA) *reinterpret_cast<float2*>(sL + i * LL + j) = make_float2(l[0], l[1]);
    }
  }
  if constexpr (DELTA) {
    __syncthreads();
    if (tid < CH) {                              // column tid of (1 + L)^-1 by forward substitution
      float x[CH];
#pragma unroll
      for (int i = 0; i < CH; ++i) x[i] = 0.f;
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        float s[4] = {i == tid ? 1.f : 0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int m = 0; m < i; m += 4) {         // L is zero on and above the diagonal
          const float4 l = *reinterpret_cast<const float4*>(sL + i * LL + m);
          s[0] -= l.x * x[m]; s[1] -= l.y * x[m + 1]; s[2] -= l.z * x[m + 2]; s[3] -= l.w * x[m + 3];
        }
        x[i] = (s[0] + s[1]) + (s[2] + s[3]);
      }
      const float beta = sB[tid];
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        bf16 hi, lo;
        split_bf16(x[i] * beta, hi, lo);
        gA[2 * TRI + i * CH + tid] = hi;
        gA[3 * TRI + i * CH + tid] = lo;
      }
    }
  }
}

struct ChunkSmem {
  int D, LD, k, q, a, v, s, stage, state, u, w, r, total;      // byte offsets inside a stage, then of the shared parts
};
__host__ __device__ inline ChunkSmem chunk_smem(int dp, bool delta) {
  ChunkSmem m;
  m.D = up16(dp); m.LD = m.D + 8;
  m.k = 0;
  m.q = m.k + CH * m.LD * 2;
  m.a = m.q + CH * m.LD * 2;
  m.v = m.a + (delta ? 4 : 2) * CH * LT * 2;
  m.s = m.v + CH * LV * 2;
  m.stage = m.s + SCALARS * 4;
  m.state = 2 * m.stage;                        // state, two parts
  m.w = m.state + 2 * m.D * LV * 2;             // U with the decay to the chunk's end, two parts
  m.u = m.w + 2 * CH * LV * 2;                  // U, two parts (delta rule)
  m.r = m.u + (delta ? 2 * CH * LV * 2 : 0);    // R, two parts (delta rule)
  m.total = m.r + (delta ? 2 * CH * LV * 2 : 0);
  return m;
}

__device__ __forceinline__ void store_split(bf16* hi_at, bf16* lo_at, float a, float b) {
  bf16 hi[2], lo[2];
  split_bf16(a, hi[0], lo[0]);
  split_bf16(b, hi[1], lo[1]);
  *reinterpret_cast<__nv_bfloat162*>(hi_at) = __nv_bfloat162(hi[0], hi[1]);
  *reinterpret_cast<__nv_bfloat162*>(lo_at) = __nv_bfloat162(lo[0], lo[1]);
}

// grid (ceil(vp / 16), heads, sequences), 256 threads: warps 0..3 own the state (16 MT rows each), warps 4..7 the output
template <bool DELTA, int MT>
__global__ void __launch_bounds__(256)
chunk_scan_kernel(const Recurrence r, const uint8_t* __restrict__ scratch, int chunks) {
  extern __shared__ __align__(16) uint8_t smem[];
  const ChunkSmem m = chunk_smem(r.dp, DELTA);
  const int v0 = blockIdx.x * VS, h = blockIdx.y, seq = blockIdx.z, kvh = h / (r.heads / r.kv_heads);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int T = r.pos.per_seq, D = m.D, LD = m.LD;
  const long long row0 = (long long)seq * T;
  bf16* sS = reinterpret_cast<bf16*>(smem + m.state);
  bf16* sW = reinterpret_cast<bf16*>(smem + m.w);
  bf16* sU = reinterpret_cast<bf16*>(smem + m.u);
  bf16* sR = reinterpret_cast<bf16*>(smem + m.r);
  const int S_LO = D * LV, T_LO = CH * LV;                       // offset of the low parts
  const bf16* act = (const bf16*)r.act;
  auto load_chunk = [&](int c) {
    uint8_t* st = smem + (c & 1) * m.stage;
    const int t0 = c * CH, n = min(CH, T - t0);
    const bf16* rows = act + (row0 + t0) * r.lda;
    bf16 *sk = reinterpret_cast<bf16*>(st + m.k), *sq = reinterpret_cast<bf16*>(st + m.q), *sa = reinterpret_cast<bf16*>(st + m.a);
    bf16* sv = reinterpret_cast<bf16*>(st + m.v);
    for (int i = tid; i < CH * (D / 8); i += 256) {
      const int row = i / (D / 8), col = (i - row * (D / 8)) * 8;
      const bool in = row < n && col < r.dp;
      const long long at = in ? row * r.lda + kvh * r.dp + col : 0;
      cp_async16_or_zero(sk + row * LD + col, rows + (in ? r.k_off : 0) + at, in);
      cp_async16_or_zero(sq + row * LD + col, rows + (in ? r.q_off : 0) + at, in);
    }
    if (tid < CH * 2) {
      const int row = tid >> 1, col = (tid & 1) * 8;
      const bool in = row < n && v0 + col < r.vp;
      cp_async16_or_zero(sv + row * LV + col, rows + (in ? row * r.lda + r.v_off + (long long)h * r.vp + v0 + col : 0), in);
    }
    const uint8_t* unit = scratch + ((long long)(seq * chunks + c) * r.heads + h) * chunk_bytes(DELTA);
    const bf16* ga = reinterpret_cast<const bf16*>(unit);
    constexpr int MATS = DELTA ? 4 : 2;
    for (int i = tid; i < CH * 8; i += 256) {
      const int row = i >> 3, col = (i & 7) * 8;
      if (col <= (row | 15)) {                                   // blocks on and below the diagonal
#pragma unroll
        for (int a = 0; a < MATS; ++a) cp_async16(sa + a * CH * LT + row * LT + col, ga + a * TRI + row * CH + col);
      }
    }
    if (tid < SCALARS / 4) cp_async16(st + m.s + tid * 16, unit + MATS * TRI * 2 + tid * 16);
    cp_async_commit();
  };
  load_chunk(0);
  float* state = r.state.ptr + seq * r.state.seq_stride + (long long)h * r.dp * r.vp + v0;
  const bool fresh = r.pos.lens[seq] == 0;
  float st[MT][2][4] = {};
  auto each_state = [&](auto f) {                                // f(row of the state, column, tile, column tile, first element)
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int half = 0; half < 2; ++half)
          f((warp + 4 * i) * 16 + (lane >> 2) + half * 8, t * 8 + (lane & 3) * 2, i, t, half * 2);
  };
  auto publish_state = [&] {
    each_state([&](int d, int v, int i, int t, int e) {
      if (d < D) store_split(sS + d * LV + v, sS + S_LO + d * LV + v, st[i][t][e], st[i][t][e + 1]);
    });
  };
  if (warp < 4) {
    each_state([&](int d, int v, int i, int t, int e) {
      const bool in = !fresh && d < r.dp && v0 + v < r.vp;
      const float2 x = in ? *reinterpret_cast<const float2*>(state + (long long)d * r.vp + v) : make_float2(0.f, 0.f);
      st[i][t][e] = x.x; st[i][t][e + 1] = x.y;
    });
    publish_state();
  }
  const int mrow = (warp & 3) * 16;                              // this warp's 16 tokens of a chunk
  const int ri = mrow + (lane >> 2), ci = (lane & 3) * 2;        // first row and column of its accumulators
  auto a_frag = [&](uint32_t (&a)[4], const bf16* tile, int ld, int k) { ldmatrix4(a, tile + (mrow + (lane & 15)) * ld + k + (lane >> 4) * 8); };
  auto b_frag = [&](uint32_t (&b)[4], const bf16* rows, int k) { ldmatrix4_trans(b, rows + (k + (lane & 15)) * LV + (lane >> 4) * 8); };
  for (int c = 0; c < chunks; ++c) {
    cp_async_wait<0>();
    __syncthreads();                                             // the chunk has arrived; the state is published; the other stage is free
    if (c + 1 < chunks) load_chunk(c + 1);
    const uint8_t* stg = smem + (c & 1) * m.stage;
    const bf16 *sk = reinterpret_cast<const bf16*>(stg + m.k), *sq = reinterpret_cast<const bf16*>(stg + m.q);
    const bf16 *sA = reinterpret_cast<const bf16*>(stg + m.a), *sT = sA + 2 * CH * LT, *sv = reinterpret_cast<const bf16*>(stg + m.v);
    const float* sc = reinterpret_cast<const float*>(stg + m.s);
    float o[2][4];
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[t][e] = 0.f;
    // K S (warps 0..3, delta rule) and Q S (warps 4..7)
    if (DELTA || warp >= 4) {
      const bf16* rows = warp < 4 ? sk : sq;
      for (int k = 0; k < D; k += 16) {
        uint32_t a[4], hi[4], lo[4];
        a_frag(a, rows, LD, k);
        b_frag(hi, sS, k);
        b_frag(lo, sS + S_LO, k);
        mma_16816(o[0], a, hi[0], hi[1]);
        mma_16816(o[1], a, hi[2], hi[3]);
        mma_16816(o[0], a, lo[0], lo[1]);
        mma_16816(o[1], a, lo[2], lo[3]);
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[t][e] *= sc[(warp < 4 ? 0 : CH) + ri + (e >> 1) * 8];
    }
    if (warp < 4) {
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = ri + half * 8, j = t * 8 + ci;
          const float2 v = unpack_bf16(*reinterpret_cast<const uint32_t*>(sv + i * LV + j));
          if (DELTA) {
            store_split(sR + i * LV + j, sR + T_LO + i * LV + j, v.x - o[t][half * 2], v.y - o[t][half * 2 + 1]);
          } else {
            const float w = sc[2 * CH + i];
            store_split(sW + i * LV + j, sW + T_LO + i * LV + j, v.x * w, v.y * w);
          }
        }
    }
    __syncthreads();
    if constexpr (DELTA) {                                       // U = T R: warp = 16 tokens x 8 columns
      const int t = warp >> 2;
      float u[4] = {0.f, 0.f, 0.f, 0.f};
      for (int k = 0; k <= mrow; k += 16) {
        uint32_t th[4], tl[4], hi[4], lo[4];
        a_frag(th, sT, LT, k);
        a_frag(tl, sT + CH * LT, LT, k);
        b_frag(hi, sR, k);
        b_frag(lo, sR + T_LO, k);
        const uint32_t h0 = t ? hi[2] : hi[0], h1 = t ? hi[3] : hi[1], l0 = t ? lo[2] : lo[0], l1 = t ? lo[3] : lo[1];
        mma_16816(u, th, h0, h1);
        mma_16816(u, tl, h0, h1);
        mma_16816(u, th, l0, l1);
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = ri + half * 8, j = t * 8 + ci;
        const float w = sc[2 * CH + i];
        store_split(sU + i * LV + j, sU + T_LO + i * LV + j, u[half * 2], u[half * 2 + 1]);
        store_split(sW + i * LV + j, sW + T_LO + i * LV + j, u[half * 2] * w, u[half * 2 + 1] * w);
      }
      __syncthreads();
    }
    if (warp >= 4) {                                             // O = decayed Q S + A U
      for (int k = 0; k <= mrow; k += 16) {
        uint32_t ah[4], al[4], hi[4];
        a_frag(ah, sA, LT, k);
        a_frag(al, sA + CH * LT, LT, k);
        b_frag(hi, DELTA ? sU : sv, k);
        mma_16816(o[0], ah, hi[0], hi[1]);
        mma_16816(o[1], ah, hi[2], hi[3]);
        mma_16816(o[0], al, hi[0], hi[1]);
        mma_16816(o[1], al, hi[2], hi[3]);
        if constexpr (DELTA) {
          uint32_t lo[4];
          b_frag(lo, sU + T_LO, k);
          mma_16816(o[0], ah, lo[0], lo[1]);
          mma_16816(o[1], ah, lo[2], lo[3]);
        }
      }
      bf16* out = (bf16*)r.o + (row0 + c * CH) * r.ldo + (long long)h * r.vp + v0;
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = ri + half * 8, j = t * 8 + ci;
          if (c * CH + i < T && v0 + j < r.vp) *reinterpret_cast<uint32_t*>(out + i * r.ldo + j) = pack_bf16(o[t][half * 2], o[t][half * 2 + 1]);
        }
    } else {                                                     // S = decayed S + K^T W
      const float g = sc[3 * CH];
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) st[i][t][e] *= g;
#pragma unroll
      for (int k = 0; k < CH; k += 16) {
        uint32_t hi[4], lo[4];
        b_frag(hi, sW, k);
        b_frag(lo, sW + T_LO, k);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          const int d0 = (warp + 4 * i) * 16;
          if (d0 < D) {
            uint32_t a[4];                                       // K^T: rows are the head's dimensions, k the tokens
            ldmatrix4_trans(a, sk + (k + (lane & 7) + (lane >> 4) * 8) * LD + d0 + ((lane >> 3) & 1) * 8);
            mma_16816(st[i][0], a, hi[0], hi[1]);
            mma_16816(st[i][1], a, hi[2], hi[3]);
            mma_16816(st[i][0], a, lo[0], lo[1]);
            mma_16816(st[i][1], a, lo[2], lo[3]);
          }
        }
      }
      publish_state();                                           // Q S and K S of this chunk have been read
    }
  }
  if (warp < 4)
    each_state([&](int d, int v, int i, int t, int e) {
      if (d < r.dp && v0 + v < r.vp) *reinterpret_cast<float2*>(state + (long long)d * r.vp + v) = make_float2(st[i][t][e], st[i][t][e + 1]);
    });
}

// ------------------------------------------------------------------------- norm, gate
struct NormGate {
  const void* o; long long ldo; const void* gate; long long ldg; const float* w; float eps;
  int rows, groups, n, np, act; float out_scale;
  void* y; long long ldy;
};
template <typename T>
__device__ __forceinline__ void gate8(const NormGate& d, float (&v)[8], long long row, int col, int c, float r) {
  float g[8], w[8];
  load8((const T*)d.gate + row * d.ldg + col, g);
  load8(d.w + c, w);
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const float a = sigmoid_of<T>(g[j]);
    v[j] *= r * w[j] * (d.act == 0 ? g[j] * a : a);
  }
  store8((T*)d.y + row * d.ldy + col, v);
}

// the last taps - 1 inputs of a sequence's convolution, token t in slot t % taps
template <typename T>
__device__ void keep_inputs(const DeltaInputs& d, int job) {
  const int back = d.taps - 1, seq = job / back, t = d.pos.per_seq - 1 - job % back;
  if (t < 0) return;
  const int channels = 2 * d.kv_heads * d.dp + d.heads * d.vp;
  const T* z = (const T*)d.z + ((long long)seq * d.pos.per_seq + t) * d.ldz;
  float* ring = d.ring.ptr + seq * d.ring.seq_stride + (long long)((d.pos.lens[seq] + t) % d.taps) * channels;
  for (int c = threadIdx.x * 8; c < channels; c += blockDim.x * 8) {
    float v[8];
    load8(z + c, v);
    store8(ring + c, v);
  }
}

// a warp per group
template <typename T>
__global__ void __launch_bounds__(256)
norm_gate_warp_kernel(const NormGate d, const DeltaInputs ring, int main_blocks) {
  if ((int)blockIdx.x >= main_blocks) return keep_inputs<T>(ring, blockIdx.x - main_blocks);
  const int lane = threadIdx.x & 31;
  const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5), row = i / d.groups;
  if (row >= d.rows) return;
  const int g0 = (int)(i - row * d.groups) * d.np;
  const T* o = (const T*)d.o + row * d.ldo + g0;
  float ss = 0.f;
  for (int c = lane * 8; c < d.np; c += 256) {
    float v[8];
    load8(o + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
  }
  const float r = inv_rms(warp_sum(ss), d.n, d.eps) * d.out_scale;
  for (int c = lane * 8; c < d.np; c += 256) {
    float v[8];
    load8(o + c, v);
    gate8<T>(d, v, row, g0 + c, c, r);
  }
}
// a block per row of one group
template <typename T>
__global__ void __launch_bounds__(256)
norm_gate_row_kernel(const NormGate d) {
  __shared__ float red[32];
  const long long row = blockIdx.x;
  const T* o = (const T*)d.o + row * d.ldo;
  float ss[1] = {0.f};
  for (int c = threadIdx.x * 8; c < d.np; c += 2048) {
    float v[8];
    load8(o + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss[0] += v[j] * v[j];
  }
  block_sum<1>(ss, red);
  const float r = inv_rms(ss[0], d.n, d.eps) * d.out_scale;
  for (int c = threadIdx.x * 8; c < d.np; c += 2048) {
    float v[8];
    load8(o + c, v);
    gate8<T>(d, v, row, c, c, r);
  }
}

bool inputs_ok(const DeltaInputs& d) {
  return d.rows > 0 && d.pos.lens && d.pos.per_seq > 0 && d.rows % d.pos.per_seq == 0 && d.heads > 0 && d.kv_heads > 0 && d.heads % d.kv_heads == 0 &&
         d.dim > 0 && d.dim <= d.dp && d.vdim > 0 && d.vdim <= d.vp && !(d.dp & 7) && !(d.vp & 7) && d.taps > 0 && !(d.ldz & 7) && d.z && d.conv &&
         d.ring.ptr && !(d.ring.seq_stride & 3) && !(d.f32 && !d.z_f32);
}
bool recurrence_ok(const Recurrence& d) {
  return d.rows > 0 && d.pos.lens && d.pos.per_seq > 0 && d.rows % d.pos.per_seq == 0 && d.rows / d.pos.per_seq <= 65535 && d.heads > 0 && d.heads <= 65535 &&
         d.kv_heads > 0 && d.heads % d.kv_heads == 0 && d.dp > 0 && d.dp <= 512 && !(d.dp & 7) && d.vp > 0 && !(d.vp & 7) && !((d.q_off | d.k_off | d.v_off) & 7) &&
         !(d.lda & 7) && !(d.ldo & 7) && d.act && d.o && d.state.ptr && !(d.state.seq_stride & 3) && (d.beta_g ? d.norms != nullptr : d.log_decay != nullptr);
}

}  // namespace

cudaError_t delta_prepare(const DeltaInputs& d, void* act, float* norms, float* beta_g, cudaStream_t s) {
  if (!inputs_ok(d) || !d.ba || d.rows / d.pos.per_seq > 65535) return cudaErrorInvalidValue;
  const dim3 grid((d.pos.per_seq + PREP_TOKENS - 1) / PREP_TOKENS, (2 * d.kv_heads + d.heads + 3) / 4, d.rows / d.pos.per_seq);
  const bool held = d.taps <= 4;
  if (d.f32) {
    auto k = held ? delta_prepare_kernel<float, float, 4> : delta_prepare_kernel<float, float, 0>;
    k<<<grid, 128, 0, s>>>(d, (float*)act, norms, beta_g);
  } else if (d.z_f32) {
    auto k = held ? delta_prepare_kernel<bf16, float, 4> : delta_prepare_kernel<bf16, float, 0>;
    k<<<grid, 128, 0, s>>>(d, (bf16*)act, norms, beta_g);
  } else {
    auto k = held ? delta_prepare_kernel<bf16, bf16, 4> : delta_prepare_kernel<bf16, bf16, 0>;
    k<<<grid, 128, 0, s>>>(d, (bf16*)act, norms, beta_g);
  }
  return cudaGetLastError();
}

cudaError_t silu_rows(bool f32, const void* z, long long ldz, int rows, int n, void* act, long long lda, cudaStream_t s) {
  if (rows <= 0 || n <= 0 || (n & 7) || (ldz & 7) || (lda & 7)) return cudaErrorInvalidValue;
  const unsigned blocks = (unsigned)(((long long)rows * (n / 8) + 255) / 256);
  if (f32) silu_rows_kernel<float><<<blocks, 256, 0, s>>>((const float*)z, ldz, rows, n, (float*)act, lda);
  else silu_rows_kernel<bf16><<<blocks, 256, 0, s>>>((const bf16*)z, ldz, rows, n, (bf16*)act, lda);
  return cudaGetLastError();
}

template <typename T, bool DELTA>
static cudaError_t launch_scan(const Recurrence& d, cudaStream_t s) {
  const dim3 grid((d.vp + 15) / 16, d.heads, d.rows / d.pos.per_seq);
  if (d.dp <= 32) recurrence_scan_kernel<T, DELTA, 1><<<grid, 128, 0, s>>>(d);
  else if (d.dp <= 64) recurrence_scan_kernel<T, DELTA, 2><<<grid, 128, 0, s>>>(d);
  else if (d.dp <= 128) recurrence_scan_kernel<T, DELTA, 4><<<grid, 128, 0, s>>>(d);
  else if (d.dp <= 256) recurrence_scan_kernel<T, DELTA, 8><<<grid, 128, 0, s>>>(d);
  else recurrence_scan_kernel<T, DELTA, 16><<<grid, 128, 0, s>>>(d);
  return cudaGetLastError();
}
cudaError_t recurrence_scan(const Recurrence& d, cudaStream_t s) {
  if (!recurrence_ok(d)) return cudaErrorInvalidValue;
  if (d.f32) return d.beta_g ? launch_scan<float, true>(d, s) : launch_scan<float, false>(d, s);
  return d.beta_g ? launch_scan<bf16, true>(d, s) : launch_scan<bf16, false>(d, s);
}

bool recurrence_chunks_supported(int dp) { return dp > 0 && dp <= 128 && !(dp & 7); }
size_t recurrence_scratch(int seqs, int per_seq, int heads, bool delta) {
  return (size_t)seqs * ((per_seq + CH - 1) / CH) * heads * chunk_bytes(delta);
}

template <bool DELTA>
static cudaError_t launch_chunks(const Recurrence& d, uint8_t* scratch, cudaStream_t s) {
  static PerDeviceOnce configured;
  constexpr int MAX_SMEM = 200 * 1024;
  cudaError_t e = configured.once([] {
    cudaError_t r = cudaFuncSetAttribute(chunk_scan_kernel<DELTA, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SMEM);
    return r != cudaSuccess ? r : cudaFuncSetAttribute(chunk_scan_kernel<DELTA, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SMEM);
  });
  if (e != cudaSuccess) return e;
  const int seqs = d.rows / d.pos.per_seq, chunks = (d.pos.per_seq + CH - 1) / CH, LD = up16(d.dp) + 8;
  const ChunkSmem m = chunk_smem(d.dp, DELTA);
  if (m.total > MAX_SMEM) return cudaErrorInvalidValue;
  const int tiles = 2 * CH * LD * 2, system = CH * (CH + 4) * 4;
  chunk_gram_kernel<DELTA><<<dim3(chunks, d.heads, seqs), 128, tiles > system ? tiles : system, s>>>(d, scratch);
  e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  const dim3 grid((d.vp + VS - 1) / VS, d.heads, seqs);
  if (m.D <= 64) chunk_scan_kernel<DELTA, 1><<<grid, 256, m.total, s>>>(d, scratch, chunks);
  else chunk_scan_kernel<DELTA, 2><<<grid, 256, m.total, s>>>(d, scratch, chunks);
  return cudaGetLastError();
}
cudaError_t recurrence_chunks(const Recurrence& d, void* scratch, cudaStream_t s) {
  if (!recurrence_ok(d) || d.f32 || !recurrence_chunks_supported(d.dp) || !scratch) return cudaErrorInvalidValue;
  return d.beta_g ? launch_chunks<true>(d, (uint8_t*)scratch, s) : launch_chunks<false>(d, (uint8_t*)scratch, s);
}

cudaError_t norm_gate(bool f32, const void* o, long long ldo, const void* gate, long long ldg, const float* w, float eps, int rows, int groups,
                      int n, int np, int act, float out_scale, void* y, long long ldy, const DeltaInputs* ring, cudaStream_t s) {
  if (rows <= 0 || groups <= 0 || n <= 0 || n > np || (np & 7) || ((ldo | ldg | ldy) & 7) || (ring && (!inputs_ok(*ring) || ring->z_f32 != f32)))
    return cudaErrorInvalidValue;
  const NormGate d{o, ldo, gate, ldg, w, eps, rows, groups, n, np, act, out_scale, y, ldy};
  if (groups == 1 && !ring) {
    if (f32) norm_gate_row_kernel<float><<<rows, 256, 0, s>>>(d);
    else norm_gate_row_kernel<bf16><<<rows, 256, 0, s>>>(d);
    return cudaGetLastError();
  }
  const int blocks = (int)(((long long)rows * groups + 7) / 8);
  const int extra = ring ? (ring->taps - 1) * (ring->rows / ring->pos.per_seq) : 0;
  const DeltaInputs in = ring ? *ring : DeltaInputs{};
  if (f32) norm_gate_warp_kernel<float><<<blocks + extra, 256, 0, s>>>(d, in, blocks);
  else norm_gate_warp_kernel<bf16><<<blocks + extra, 256, 0, s>>>(d, in, blocks);
  return cudaGetLastError();
}

}  // namespace serve
}  // namespace nc
