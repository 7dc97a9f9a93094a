// Recurrences over a per-sequence state (dp x vp floats a head): the gated delta rule and linear attention with a fixed
// decay per head, for portions of several tokens.
//
//   prepare           short convolution + silu of queries, keys and values (fixed decay: silu alone), inverse norms, step
//                     sizes, log decays; as rows for the token-by-token kernel or as the chunk kernels' tiles
//   recurrence_scan   token by token, the state in registers: float, short portions, wide heads
//   recurrence_chunks chunks of 64 tokens, two kernels:
//       gram   (parallel over chunks) A = (Q K^T) with decays, causal; for the delta rule also the inverse of the unit
//              triangular system that the tokens of a chunk solve, T = (1 + strict(beta K K^T with decays))^-1 beta
//       scan   (sequential over chunks, one CTA per 16 state columns)
//                 R = V - decayed K S,  U = T R        delta rule;   U = V  fixed decay
//                 O = decayed Q S + A U
//                 S = decayed S + K^T (decayed U)
//              One warp copies whole chunks into shared memory, four follow the state from chunk to chunk, four more
//              read it out behind them.
//   norm_gate         RMS norm and gate of what a recurrence read out, and the convolution's last inputs
//
// Exactness: the products run on bf16 operands, so every operand that is a float (S, T, A, U, R) enters as the sum of two bf16
// values, and what scales rows (inverse norms, decays) is applied to accumulators, not to operands: keys, queries and values are
// the bf16 activations themselves. The state is float from chunk to chunk, and a read-out that nearly cancels keeps its digits.
#include <type_traits>

#include "mma.cuh"

namespace nc {
namespace serve {

namespace {

template <typename T> __device__ __forceinline__ float silu_of(float v) { return v * sigmoid_of<T>(v); }

// four neighbouring values as they lie in memory
template <typename T> struct Raw4;
template <> struct Raw4<float> {
  float4 a;
  __device__ void load(const float* p) { a = *reinterpret_cast<const float4*>(p); }
  __device__ void set(const float (&f)[4]) { a = make_float4(f[0], f[1], f[2], f[3]); }
  __device__ void get(float (&f)[4]) const { f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; }
};
template <> struct Raw4<bf16> {
  uint2 u;
  __device__ void load(const bf16* p) { u = *reinterpret_cast<const uint2*>(p); }
  __device__ void set(const float (&f)[4]) { u = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3])); }
  __device__ void get(float (&f)[4]) const {
    const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
};

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

// ------------------------------------------------------------------------------ tiles
constexpr int CH = 64;                       // tokens per chunk
// A lower triangular 64 x 64 operand: four bands of 16 rows, band b with its first 16 (b + 1) columns and a pitch of 8 more.
__host__ __device__ constexpr int band_pitch(int b) { return 16 * (b + 1) + 8; }
__host__ __device__ constexpr int band_at(int b) { return 16 * (8 * b * (b + 1) + 8 * b); }
constexpr int MAT = band_at(4);
__device__ __forceinline__ int band_index(int i, int j) { return band_at(i >> 4) + (i & 15) * band_pitch(i >> 4) + j; }
constexpr int SCALARS = 200;                 // floats per chunk and head: three vectors of 64, the chunk's total decay, padding
constexpr int VS = 16;                       // state columns per CTA
constexpr int LV = VS + 8;

__host__ __device__ constexpr int tile_dim(int dp) { return dp <= 64 ? 64 : 128; }          // columns of a q or k tile
// Tiles of a portion, bf16: per (sequence, chunk, key head) q then k, 64 x (D + 8); behind them per (sequence, chunk, head,
// slice of 16 columns) v, 64 x 24. Rows past the portion and columns past a head are zero, the pitch's padding is anything.
struct Tiles {
  int chunks, D, slices;
  long long qk_unit, v_unit, v_base;         // elements
  __host__ __device__ Tiles(int seqs, int per_seq, int heads, int kv_heads, int dp, int vp) {
    chunks = (per_seq + CH - 1) / CH;
    D = tile_dim(dp);
    slices = (vp + VS - 1) / VS;
    qk_unit = 2ll * CH * (D + 8);
    v_unit = (long long)CH * LV;
    v_base = (long long)seqs * chunks * kv_heads * qk_unit;
  }
  __host__ __device__ long long elements(int seqs, int heads) const { return v_base + (long long)seqs * chunks * heads * slices * v_unit; }
};
__host__ __device__ constexpr size_t chunk_bytes(bool delta) { return (size_t)(delta ? 4 : 2) * MAT * 2 + SCALARS * 4; }

// ---------------------------------------------------------------------------- prepare
constexpr int PREP_TOKENS = 8;         // tokens a warp walks through

// grid (token groups of a sequence, ceil(jobs / 4), sequences), a warp per job: query heads, key heads, value heads.
// TAPS > 0: at most TAPS taps, the inputs stay in registers; 0: any number, re-read; -1: no convolution and no norms
// (fixed decay). TILES: out is laid out as Tiles, otherwise rows x channels.
template <typename T, typename TZ, int TAPS, bool TILES>
__global__ void __launch_bounds__(128, sizeof(TZ) == 2 ? 6 : 4)
prepare_kernel(const DeltaInputs d, T* __restrict__ out, float* __restrict__ norms, float* __restrict__ beta_g) {
  const int lane = threadIdx.x & 31, job = blockIdx.y * 4 + (threadIdx.x >> 5);
  const int G = d.kv_heads, H = d.heads, per_seq = d.pos.per_seq, seq = blockIdx.z;
  if (job >= 2 * G + H) return;
  const int t0 = blockIdx.x * PREP_TOKENS, n = min(PREP_TOKENS, per_seq - t0);      // n <= 0: only zeros to write
  const int channels = 2 * G * d.dp + H * d.vp, size = job < 2 * G ? d.dp : d.vp;
  const int ch0 = job < 2 * G ? job * d.dp : 2 * G * d.dp + (job - 2 * G) * d.vp;
  const int start = TAPS >= 0 ? d.pos.lens[seq] : 0;
  const long long row0 = (long long)seq * per_seq;
  const float* ring = TAPS >= 0 ? d.ring.ptr + seq * d.ring.seq_stride : nullptr;
  const Tiles tiles(gridDim.z, per_seq, H, G, d.dp, d.vp);
  auto fetch = [&](int t, int ch, float (&x)[4]) {
    if (t >= 0) {
      load4((const TZ*)d.z + (row0 + t) * d.ldz + ch, x);
    } else if (start + t >= 0) {
      load4(ring + (long long)((start + t) % d.taps) * channels + ch, x);
    } else {
      x[0] = x[1] = x[2] = x[3] = 0.f;
    }
  };
  // where the head's columns of the group's first token go, and from one token to the next
  const long long unit = (long long)seq * tiles.chunks + t0 / CH;
  const int r0 = t0 % CH;
  T* dst = !TILES ? out + (row0 + t0) * channels + ch0
           : job < 2 * G ? out + (unit * G + job % G) * tiles.qk_unit + ((job >= G ? CH : 0) + r0) * (tiles.D + 8)
                         : out + tiles.v_base + (unit * H + job - 2 * G) * tiles.slices * tiles.v_unit + r0 * LV;
  const int step = !TILES ? channels : job < 2 * G ? tiles.D + 8 : LV;
  float ss[PREP_TOKENS];
#pragma unroll
  for (int t = 0; t < PREP_TOKENS; ++t) ss[t] = 0.f;
  const int columns = !TILES ? size : job < 2 * G ? tiles.D : tiles.slices * VS;
  constexpr int BACK = TAPS > 0 ? TAPS - 1 : 0;
  const bool inside = t0 >= BACK && n == PREP_TOKENS;   // every input is a row of this portion
  for (int c = lane * 4; c < columns; c += 128) {
    const int ch = ch0 + c;
    float w[BACK + 1][4];
    Raw4<TZ> x[PREP_TOKENS + BACK];                     // x[BACK + t]: token t of the group (the ring holds what z held)
    const bool in = c < size;
    if (TAPS != 0 && inside && in) {
      const TZ* src = (const TZ*)d.z + (row0 + t0 - BACK) * d.ldz + ch;
#pragma unroll
      for (int t = 0; t < PREP_TOKENS + BACK; ++t) x[t].load(src + t * d.ldz);
    } else {
#pragma unroll
      for (int t = 0; t < PREP_TOKENS + BACK; ++t) {
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        if (in && TAPS != 0 && t - BACK < n && (t >= BACK || BACK - t < d.taps)) fetch(t0 + t - BACK, ch, f);
        x[t].set(f);
      }
    }
    if (TAPS > 0) {
#pragma unroll
      for (int i = 0; i <= BACK; ++i) {                 // tap i meets the token i places back
        if (in && i < d.taps) {
          load4(d.conv + (long long)(d.taps - 1 - i) * channels + ch, w[i]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j) w[i][j] = 0.f;
        }
      }
    }
    T* at = TILES && job >= 2 * G ? dst + (c / VS) * tiles.v_unit + c % VS : dst + c;
#pragma unroll
    for (int t = 0; t < PREP_TOKENS; ++t) {
      if (!TILES && t >= n) break;
      float a[4] = {0.f, 0.f, 0.f, 0.f};
      if (TAPS > 0) {
#pragma unroll
        for (int i = 0; i <= BACK; ++i) {
          float f[4];
          x[BACK + t - i].get(f);
#pragma unroll
          for (int j = 0; j < 4; ++j) a[j] += w[i][j] * f[j];
        }
      } else if (TAPS == 0) {
        for (int i = 0; in && t < n && i < d.taps; ++i) {
          float wi[4], xi[4];
          load4(d.conv + (long long)(d.taps - 1 - i) * channels + ch, wi);
          fetch(t0 + t - i, ch, xi);
#pragma unroll
          for (int j = 0; j < 4; ++j) a[j] += wi[j] * xi[j];
        }
      } else {
        x[t].get(a);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        a[j] = t < n ? to_f(from_f<T>(silu_of<T>(a[j]))) : 0.f;     // the norm is that of the vector that is stored
        ss[t] += a[j] * a[j];
      }
      store4(at + t * step, a);
    }
  }
  if (TAPS < 0) return;
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
    float* bg = beta_g + (row0 + t0 + lane) * 2 * H;
    bg[h] = sigmoidf(in[h]);
    bg[H + h] = d.neg_a[h] * (a > 20.f ? a : log1pf(expf(a)));
  }
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
__device__ __forceinline__ void store_split(bf16* hi_at, bf16* lo_at, float a, float b) {
  bf16 hi[2], lo[2];
  split_bf16(a, hi[0], lo[0]);
  split_bf16(b, hi[1], lo[1]);
  *reinterpret_cast<__nv_bfloat162*>(hi_at) = __nv_bfloat162(hi[0], hi[1]);
  *reinterpret_cast<__nv_bfloat162*>(lo_at) = __nv_bfloat162(lo[0], lo[1]);
}

// Two neighbouring entries (r, c), (r, c + 1) of the product of two 16 x 16 blocks in shared memory.
constexpr int LL = CH + 4;
__device__ __forceinline__ void block_dot(const float* a, const float* b, int lda, int ldb, int r, int c, float (&s)[2]) {
#pragma unroll
  for (int k = 0; k < 16; k += 4) {
    const float4 l = *reinterpret_cast<const float4*>(a + r * lda + k);
    const float lk[4] = {l.x, l.y, l.z, l.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 x = *reinterpret_cast<const float2*>(b + (k + e) * ldb + c);
      s[0] += lk[e] * x.x;
      s[1] += lk[e] * x.y;
    }
  }
}
// X = (1 + L)^-1 for a strictly lower triangular L, both 64 x LL floats; blocks of 16: the diagonal ones by forward
// substitution, the others below them from the left. All 256 threads call it; L has been written and synchronised.
__device__ void invert_unit_lower(const float* L, float* X, float (*P)[16][20]) {
  const int tid = threadIdx.x;
  if (tid < CH) {
    const int b = tid & ~15, j = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float s[2] = {i == j ? 1.f : 0.f, 0.f};
#pragma unroll
      for (int m = 0; m < i; ++m) s[m & 1] -= L[(b + i) * LL + b + m] * x[m];
      x[i] = s[0] + s[1];
      X[(b + i) * LL + b + j] = x[i];
    }
  }
  __syncthreads();
  const int half = tid >> 7, r = (tid & 127) >> 3, c = (tid & 7) * 2;      // each half takes every other block
#pragma unroll 1
  for (int d = 1; d < 4; ++d) {
#pragma unroll 1
    for (int i = d + half; i < 4; i += 2) {              // P = sum over the blocks between of L_im X_mj, j = i - d
      float s[2] = {0.f, 0.f};
      for (int m = i - d; m < i; ++m) block_dot(L + i * 16 * LL + m * 16, X + m * 16 * LL + (i - d) * 16, LL, LL, r, c, s);
      *reinterpret_cast<float2*>(&P[i - d][r][c]) = make_float2(s[0], s[1]);
    }
    __syncthreads();
#pragma unroll 1
    for (int i = d + half; i < 4; i += 2) {
      float s[2] = {0.f, 0.f};
      block_dot(X + i * 16 * LL + i * 16, &P[i - d][0][0], LL, 20, r, c, s);
      *reinterpret_cast<float2*>(X + (i * 16 + r) * LL + (i - d) * 16 + c) = make_float2(-s[0], -s[1]);
    }
    __syncthreads();
  }
}

// grid (chunks, heads, sequences), 256 threads: warp w has 16 tokens and every other pair of 8-key tiles. Row i of a chunk: scalars [0, 64) decayed 1/|k|, [64, 128) decayed 1/|q|,
// [128, 192) 1/|k| times the decay from the token to the chunk's end, [192] the decay over the whole chunk.
template <bool DELTA, int D>
__global__ void __launch_bounds__(256)
chunk_gram_kernel(const Recurrence r, uint8_t* __restrict__ scratch) {
  constexpr int LD = D + 8, TILE = CH * LD, SYSTEM = 2 * CH * LL * 4;
  constexpr int BYTES = 2 * TILE * 2 > SYSTEM || !DELTA ? 2 * TILE * 2 : SYSTEM;
  __shared__ __align__(16) uint8_t smem[BYTES];
  __shared__ float sB[CH], sRk[CH], sRq[CH], sP[DELTA ? 3 : 1][16][20];
  __shared__ double sG[CH];                                  // log decay from the chunk's start, each token's own included
  const int chunk = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, kvh = h / (r.heads / r.kv_heads);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n = min(CH, r.pos.per_seq - chunk * CH);
  const long long row0 = (long long)seq * r.pos.per_seq + chunk * CH;
  const bf16* sQ = reinterpret_cast<const bf16*>(smem);
  const bf16* sK = sQ + TILE;
  float* sL = reinterpret_cast<float*>(smem);                // take the place of the tiles once they have been used
  float* sX = sL + CH * LL;
  const Tiles tiles(gridDim.z, r.pos.per_seq, r.heads, r.kv_heads, r.dp, r.vp);
  const uint8_t* src = reinterpret_cast<const uint8_t*>((const bf16*)r.act + (((long long)seq * tiles.chunks + chunk) * r.kv_heads + kvh) * tiles.qk_unit);
#pragma unroll
  for (int i = tid * 16; i < 2 * TILE * 2; i += 256 * 16) cp_async16(smem + i, src + i);
  cp_async_commit();
  uint8_t* unit = scratch + ((long long)(seq * gridDim.x + chunk) * r.heads + h) * chunk_bytes(DELTA);
  bf16* gA = reinterpret_cast<bf16*>(unit);
  float* gS = reinterpret_cast<float*>(unit + (DELTA ? 4 : 2) * MAT * 2);
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
  const int mt = warp & 3, odd = warp >> 2;
  float qk[4][4], kk[DELTA ? 4 : 1][4];                         // tile u: keys (2 (u / 2) + odd) * 16 + (u % 2) * 8 ...
#pragma unroll
  for (int t = 0; t < 4; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) { qk[t][e] = 0.f; if (DELTA) kk[t][e] = 0.f; }
#pragma unroll
  for (int k = 0; k < D; k += 16) {
    uint32_t aq[4], ak[4];
    ldmatrix4(aq, sQ + (mt * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
    if (DELTA) ldmatrix4(ak, sK + (mt * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int j0 = (2 * u + odd) * 16;
      if (j0 > mt * 16) break;                                  // blocks above the diagonal are never read
      uint32_t b[4];                                            // 16 keys, both halves of k
      ldmatrix4(b, sK + (j0 + (lane & 7) + (lane >> 4) * 8) * LD + k + ((lane >> 3) & 1) * 8);
      mma_16816(qk[2 * u], aq, b[0], b[1]);
      mma_16816(qk[2 * u + 1], aq, b[2], b[3]);
      if constexpr (DELTA) {
        mma_16816(kk[2 * u], ak, b[0], b[1]);
        mma_16816(kk[2 * u + 1], ak, b[2], b[3]);
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    const int j0 = (2 * (u >> 1) + odd) * 16;
    if (j0 > mt * 16) break;
    const int j = j0 + (u & 1) * 8 + (lane & 3) * 2;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = mt * 16 + (lane >> 2) + half * 8;
      float a[2], l[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = j + e;
        const float decay = c <= i ? expf((float)(sG[i] - sG[c])) : 0.f;
        a[e] = c <= i ? sRq[i] * sRk[c] * decay * qk[u][half * 2 + e] : 0.f;
        if constexpr (DELTA) l[e] = c < i ? sB[i] * sRk[i] * sRk[c] * decay * kk[u][half * 2 + e] : 0.f;
      }
      store_split(gA + band_index(i, j), gA + MAT + band_index(i, j), a[0], a[1]);
      if constexpr (DELTA) *reinterpret_cast<float2*>(sL + i * LL + j) = make_float2(l[0], l[1]);
    }
  }
  if constexpr (DELTA) {
    __syncthreads();
    invert_unit_lower(sL, sX, sP);
    for (int e = tid; e < CH * CH / 2; e += 256) {
      const int i = e / (CH / 2), j = (e % (CH / 2)) * 2;
      if (j > (i | 15)) continue;
      const bool diagonal = (i >> 4) == (j >> 4);               // the substitution leaves zeros above the diagonal
      const float2 x = *reinterpret_cast<const float2*>(sX + i * LL + j);
      store_split(gA + 2 * MAT + band_index(i, j), gA + 3 * MAT + band_index(i, j), diagonal && j > i ? 0.f : x.x * sB[j], diagonal && j + 1 > i ? 0.f : x.y * sB[j + 1]);
    }
  }
}

// Shared memory of the scan: three stages of a chunk's operands, then what the warps hand each other.
constexpr int STAGES = 3;
template <bool DELTA, int D>
struct ScanSmem {
  static constexpr int LD = D + 8, MATS = DELTA ? 4 : 2;
  static constexpr int QK_BYTES = 2 * CH * LD * 2, UNIT_BYTES = MATS * MAT * 2 + SCALARS * 4, V_BYTES = CH * LV * 2;
  static constexpr int Q = 0, K = CH * LD * 2, A = QK_BYTES, SC = A + MATS * MAT * 2, V = A + UNIT_BYTES;
  static constexpr int STAGE = QK_BYTES + UNIT_BYTES + V_BYTES;
  static constexpr int PART = CH * LV, S_PART = D * LV;         // elements of one part (high or low) of a 64 x 16 operand, of the state
  static constexpr int S = STAGES * STAGE;                      // state
  static constexpr int W = S + 2 * S_PART * 2;                  // U with the decay to the chunk's end
  static constexpr int R = W + 2 * PART * 2;                    // delta rule: R, then U in two buffers
  static constexpr int U = R + (DELTA ? 2 * PART * 2 : 0);
  static constexpr int BAR = U + (DELTA ? 4 * PART * 2 : 0);
  static constexpr int TOTAL = BAR + 128;
  static_assert(STAGE % 16 == 0 && TOTAL <= 227 * 1024, "stages must fit shared memory");
};

constexpr int SCAN_THREADS = 9 * 32;
// grid (ceil(vp / 16), heads, sequences): warps 0..3 own the state (16 D / 64 rows each), 4..7 the output, 8 copies. Shared
// memory bandwidth and the latency of its loads set the pace, so a product requests all its fragments before the first use.
// A wait that runs out raises the status and the kernel runs on without waiting, so that no barrier is left short.
template <bool DELTA, int D>
__global__ void __launch_bounds__(SCAN_THREADS)
chunk_scan_kernel(const Recurrence r, const uint8_t* __restrict__ scratch, int* status) {
  using M = ScanSmem<DELTA, D>;
  constexpr int LD = M::LD, MT = D / 64;                         // MT: 16-row tiles of the state a warp holds
  extern __shared__ __align__(128) uint8_t smem[];
  const int slice = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, kvh = h / (r.heads / r.kv_heads), v0 = slice * VS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int T = r.pos.per_seq;
  const Tiles tiles(gridDim.z, T, r.heads, r.kv_heads, r.dp, r.vp);
  const int chunks = tiles.chunks;
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + M::BAR);       // per stage: a chunk has arrived, has been used
  uint64_t* empty = full + STAGES;
  uint64_t *s_ready = empty + STAGES, *s_read = s_ready + 1;         // the state is published, has been read by the output warps
  uint64_t *u_ready = s_read + 1, *u_read = u_ready + 2;             // [2] U is there, has been read, by chunk parity
  volatile int* abort_flag = reinterpret_cast<volatile int*>(u_read + 2);
  if (tid == 0) {
    for (int i = 0; i < STAGES; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], 8); }
    mbar_init(s_ready, 4); mbar_init(s_read, 4);
    for (int i = 0; i < 2; ++i) { mbar_init(&u_ready[i], 4); mbar_init(&u_read[i], 4); }
    *abort_flag = 0;
    fence_mbar_init();
  }
  __syncthreads();
  auto wait = [&](uint64_t* bar, int n, int code) { mbar_wait(bar, n & 1, abort_flag, status, code, 0x5c0); };    // its n-th completion
  auto arrive = [&](uint64_t* bar) { __syncwarp(); if (lane == 0) mbar_arrive(bar); };
  auto state_sync = [] { asm volatile("bar.sync 1, 128;" ::: "memory"); };
  const int band = warp & 3, mrow = band * 16;                   // this warp's 16 tokens of a chunk
  const int ri = mrow + (lane >> 2), ci = (lane & 3) * 2;        // first row and column of its accumulators
  auto a_frag = [&](uint32_t (&a)[4], const bf16* tile, int k) { ldmatrix4(a, tile + (mrow + (lane & 15)) * LD + k + (lane >> 4) * 8); };
  auto tri_frag = [&](uint32_t (&a)[4], const bf16* mat, int k) { ldmatrix4(a, mat + band_at(band) + (lane & 15) * band_pitch(band) + k + (lane >> 4) * 8); };
  auto b_frag = [&](uint32_t (&b)[4], const bf16* rows, int k) { ldmatrix4_trans(b, rows + (k + (lane & 15)) * LV + (lane >> 4) * 8); };
  auto add = [](float (&a)[4], const float (&b)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) a[e] += b[e];
  };
  // 16 tokens x 16 columns of X S, X the chunk's queries or keys
  auto times_state = [&](float (&o)[2][4], const bf16* rows, const bf16* s) {
    constexpr int HALF = D / 32;                                 // k-steps in flight
    float lo[2][4] = {};
#pragma unroll
    for (int k0 = 0; k0 < D; k0 += HALF * 16) {
      uint32_t a[HALF][4], bh[HALF][4], bl[HALF][4];
#pragma unroll
      for (int k = 0; k < HALF; ++k) {
        a_frag(a[k], rows, k0 + k * 16);
        b_frag(bh[k], s, k0 + k * 16);
        b_frag(bl[k], s + M::S_PART, k0 + k * 16);
      }
#pragma unroll
      for (int k = 0; k < HALF; ++k) {
        mma_16816(o[0], a[k], bh[k][0], bh[k][1]);
        mma_16816(o[1], a[k], bh[k][2], bh[k][3]);
        mma_16816(lo[0], a[k], bl[k][0], bl[k][1]);
        mma_16816(lo[1], a[k], bl[k][2], bl[k][3]);
      }
    }
    add(o[0], lo[0]);
    add(o[1], lo[1]);
  };
  // o += M X for a lower triangular M in two parts and a 64 x 16 X in one or two
  auto times_lower = [&](float (&o)[2][4], const bf16* m, const bf16* x, auto two_parts) {
    constexpr bool TWO = decltype(two_parts)::value;
    uint32_t ah[4][4], al[4][4], bh[4][4], bl[TWO ? 4 : 1][4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (k > band) break;
      tri_frag(ah[k], m, k * 16);
      b_frag(bh[k], x, k * 16);
      tri_frag(al[k], m + MAT, k * 16);
      if constexpr (TWO) b_frag(bl[k], x + M::PART, k * 16);
    }
    float p[2][4] = {}, q[2][4] = {};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (k > band) break;
      mma_16816(o[0], ah[k], bh[k][0], bh[k][1]);
      mma_16816(o[1], ah[k], bh[k][2], bh[k][3]);
      mma_16816(p[0], al[k], bh[k][0], bh[k][1]);
      mma_16816(p[1], al[k], bh[k][2], bh[k][3]);
      if constexpr (TWO) {
        mma_16816(q[0], ah[k], bl[k][0], bl[k][1]);
        mma_16816(q[1], ah[k], bl[k][2], bl[k][3]);
      }
    }
#pragma unroll
    for (int t = 0; t < 2; ++t) {
      add(o[t], p[t]);
      if constexpr (TWO) add(o[t], q[t]);
    }
  };

  if (warp == 8) {                                               // ---- copies
    if (lane == 0) {
      const bf16* qk = (const bf16*)r.act + ((long long)seq * chunks * r.kv_heads + kvh) * tiles.qk_unit;
      const bf16* v = (const bf16*)r.act + tiles.v_base + (((long long)seq * chunks * r.heads + h) * tiles.slices + slice) * tiles.v_unit;
      const uint8_t* unit = scratch + ((long long)seq * chunks * r.heads + h) * chunk_bytes(DELTA);
      for (int c = 0; c < chunks && !*abort_flag; ++c) {
        const int b = c % STAGES;
        uint8_t* st = smem + b * M::STAGE;
        if (c >= STAGES) wait(&empty[b], c / STAGES - 1, ST_WAIT_EMPTY);
        if (*abort_flag) break;
        mbar_arrive_expect_tx(&full[b], M::STAGE);
        bulk_load_1d(st + M::Q, qk + (long long)c * r.kv_heads * tiles.qk_unit, M::QK_BYTES, &full[b]);
        bulk_load_1d(st + M::A, unit + (long long)c * r.heads * chunk_bytes(DELTA), M::UNIT_BYTES, &full[b]);
        bulk_load_1d(st + M::V, v + (long long)c * r.heads * tiles.slices * tiles.v_unit, M::V_BYTES, &full[b]);
      }
    }
  } else if (warp < 4) {                                         // ---- state
    bf16* sW = reinterpret_cast<bf16*>(smem + M::W);
    bf16* sR = reinterpret_cast<bf16*>(smem + M::R);
    bf16* sS = reinterpret_cast<bf16*>(smem + M::S);
    float* state = r.state.ptr + seq * r.state.seq_stride + (long long)h * r.dp * r.vp + v0;
    const bool fresh = r.pos.lens[seq] == 0;
    float st[MT][2][4] = {};
    auto each_state = [&](auto f) {                              // f(row of the state, column, tile, column tile, first element)
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int half = 0; half < 2; ++half) f((warp + 4 * i) * 16 + (lane >> 2) + half * 8, t * 8 + ci, i, t, half * 2);
    };
    auto publish_state = [&] {
      each_state([&](int d, int v, int i, int t, int e) { store_split(sS + d * LV + v, sS + M::S_PART + d * LV + v, st[i][t][e], st[i][t][e + 1]); });
      arrive(s_ready);
    };
    each_state([&](int d, int v, int i, int t, int e) {
      const bool in = !fresh && d < r.dp && v0 + v < r.vp;
      const float2 x = in ? *reinterpret_cast<const float2*>(state + (long long)d * r.vp + v) : make_float2(0.f, 0.f);
      st[i][t][e] = x.x; st[i][t][e + 1] = x.y;
    });
    publish_state();
    state_sync();
    for (int c = 0; c < chunks; ++c) {
      const int stage = c % STAGES;
      const uint8_t* stg = smem + stage * M::STAGE;
      const bf16 *sk = reinterpret_cast<const bf16*>(stg + M::K), *sv = reinterpret_cast<const bf16*>(stg + M::V);
      const float* sc = reinterpret_cast<const float*>(stg + M::SC);
      wait(&full[stage], c / STAGES, ST_WAIT_FULL);
      uint32_t kt[MT][4][4];                                     // K^T: rows are the head's dimensions, k the tokens
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k)
          ldmatrix4_trans(kt[i][k], sk + (k * 16 + (lane & 7) + (lane >> 4) * 8) * LD + (warp + 4 * i) * 16 + ((lane >> 3) & 1) * 8);
      const float g = sc[3 * CH], w[2] = {sc[2 * CH + ri], sc[2 * CH + ri + 8]};
      float2 v[2][2];
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int half = 0; half < 2; ++half) v[t][half] = unpack_bf16(*reinterpret_cast<const uint32_t*>(sv + (ri + half * 8) * LV + t * 8 + ci));
      if constexpr (DELTA) {
        bf16* sU = reinterpret_cast<bf16*>(smem + M::U) + (c & 1) * 2 * M::PART;
        const float f[2] = {sc[ri], sc[ri + 8]};
        float x[2][4] = {};
        times_state(x, sk, sS);
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int at = (ri + half * 8) * LV + t * 8 + ci;
            store_split(sR + at, sR + M::PART + at, v[t][half].x - f[half] * x[t][half * 2], v[t][half].y - f[half] * x[t][half * 2 + 1]);
          }
        state_sync();
        float u[2][4] = {};
        times_lower(u, reinterpret_cast<const bf16*>(stg + M::A) + 2 * MAT, sR, std::true_type{});
        if (c >= 2) wait(&u_read[c & 1], (c >> 1) - 1, ST_WAIT_PEER);      // chunk c - 2 has been read out of this buffer
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int at = (ri + half * 8) * LV + t * 8 + ci;
            store_split(sW + at, sW + M::PART + at, u[t][half * 2] * w[half], u[t][half * 2 + 1] * w[half]);
            store_split(sU + at, sU + M::PART + at, u[t][half * 2], u[t][half * 2 + 1]);
          }
        arrive(&u_ready[c & 1]);
      } else {
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int at = (ri + half * 8) * LV + t * 8 + ci;
            store_split(sW + at, sW + M::PART + at, v[t][half].x * w[half], v[t][half].y * w[half]);
          }
      }
      state_sync();
      uint32_t wh[4][4], wl[4][4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        b_frag(wh[k], sW, k * 16);
        b_frag(wl[k], sW + M::PART, k * 16);
      }
      arrive(&empty[stage]);
      float lo[MT][2][4] = {};
#pragma unroll
      for (int i = 0; i < MT; ++i)                               // S = decayed S + K^T W
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) st[i][t][e] *= g;
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_16816(st[i][0], kt[i][k], wh[k][0], wh[k][1]);
          mma_16816(st[i][1], kt[i][k], wh[k][2], wh[k][3]);
          mma_16816(lo[i][0], kt[i][k], wl[k][0], wl[k][1]);
          mma_16816(lo[i][1], kt[i][k], wl[k][2], wl[k][3]);
        }
#pragma unroll
      for (int i = 0; i < MT; ++i) { add(st[i][0], lo[i][0]); add(st[i][1], lo[i][1]); }
      if (c + 1 < chunks) {
        wait(s_read, c, ST_WAIT_PEER);
        publish_state();
        state_sync();
      }
    }
    each_state([&](int d, int v, int i, int t, int e) {
      if (d < r.dp && v0 + v < r.vp) *reinterpret_cast<float2*>(state + (long long)d * r.vp + v) = make_float2(st[i][t][e], st[i][t][e + 1]);
    });
  } else {                                                       // ---- output
    for (int c = 0; c < chunks; ++c) {
      const int stage = c % STAGES;
      const uint8_t* stg = smem + stage * M::STAGE;
      const float* sc = reinterpret_cast<const float*>(stg + M::SC);
      wait(&full[stage], c / STAGES, ST_WAIT_FULL);
      wait(s_ready, c, ST_WAIT_PEER);
      float o[2][4] = {};
      times_state(o, reinterpret_cast<const bf16*>(stg + M::Q), reinterpret_cast<const bf16*>(smem + M::S));
      arrive(s_read);
      const float q[2] = {sc[CH + ri], sc[CH + ri + 8]};
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[t][e] *= q[e >> 1];
      const bf16* sA = reinterpret_cast<const bf16*>(stg + M::A);
      if constexpr (DELTA) {
        wait(&u_ready[c & 1], c >> 1, ST_WAIT_PEER);
        times_lower(o, sA, reinterpret_cast<const bf16*>(smem + M::U) + (c & 1) * 2 * M::PART, std::true_type{});
        arrive(&u_read[c & 1]);
      } else {
        times_lower(o, sA, reinterpret_cast<const bf16*>(stg + M::V), std::false_type{});
      }
      arrive(&empty[stage]);
      bf16* out = (bf16*)r.o + ((long long)seq * T + c * CH) * r.ldo + (long long)h * r.vp + v0;
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = ri + half * 8, j = t * 8 + ci;
          if (c * CH + i < T && v0 + j < r.vp) *reinterpret_cast<uint32_t*>(out + i * r.ldo + j) = pack_bf16(o[t][half * 2], o[t][half * 2 + 1]);
        }
    }
  }
  __syncthreads();
  if (*abort_flag) {                                             // copies still in flight
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
  }
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

// LANES lanes per group
template <typename T, int LANES>
__global__ void __launch_bounds__(256)
norm_gate_warp_kernel(const NormGate d, const DeltaInputs ring, int main_blocks) {
  if ((int)blockIdx.x >= main_blocks) return keep_inputs<T>(ring, blockIdx.x - main_blocks);
  const int lane = threadIdx.x % LANES;
  const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) / LANES, row = i / d.groups;
  const bool on = row < d.rows;
  const int g0 = on ? (int)(i - row * d.groups) * d.np : 0;
  const T* o = (const T*)d.o + (on ? row * d.ldo + g0 : 0);
  float ss = 0.f, first[8];
  for (int c = lane * 8; on && c < d.np; c += LANES * 8) {
    float v[8];
    load8(o + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) { ss += v[j] * v[j]; if (c < LANES * 8) first[j] = v[j]; }
  }
#pragma unroll
  for (int s = LANES / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!on) return;
  const float r = inv_rms(ss, d.n, d.eps) * d.out_scale;
  for (int c = lane * 8; c < d.np; c += LANES * 8) {
    float v[8];
    if (c < LANES * 8) {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = first[j];
    } else {
      load8(o + c, v);
    }
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

bool sizes_ok(const DeltaInputs& d) {
  return d.rows > 0 && d.pos.per_seq > 0 && d.rows % d.pos.per_seq == 0 && d.rows / d.pos.per_seq <= 65535 && d.heads > 0 && d.kv_heads > 0 &&
         d.heads % d.kv_heads == 0 && d.dp > 0 && d.vp > 0 && !(d.dp & 7) && !(d.vp & 7) && !(d.ldz & 7) && d.z && !(d.f32 && !d.z_f32);
}
bool inputs_ok(const DeltaInputs& d) {
  return sizes_ok(d) && d.pos.lens && d.dim > 0 && d.dim <= d.dp && d.vdim > 0 && d.vdim <= d.vp && d.taps > 0 && d.conv && d.ring.ptr && !(d.ring.seq_stride & 3);
}
bool recurrence_ok(const Recurrence& d) {
  return d.rows > 0 && d.pos.lens && d.pos.per_seq > 0 && d.rows % d.pos.per_seq == 0 && d.rows / d.pos.per_seq <= 65535 && d.heads > 0 && d.heads <= 65535 &&
         d.kv_heads > 0 && d.heads % d.kv_heads == 0 && d.dp > 0 && d.dp <= 512 && !(d.dp & 7) && d.vp > 0 && !(d.vp & 7) && !((d.q_off | d.k_off | d.v_off) & 7) &&
         !(d.lda & 7) && !(d.ldo & 7) && d.act && d.o && d.state.ptr && !(d.state.seq_stride & 3) && (d.beta_g ? d.norms != nullptr : d.log_decay != nullptr);
}

template <typename T, typename TZ, bool TILES>
cudaError_t launch_prepare(const DeltaInputs& d, void* out, float* norms, float* beta_g, cudaStream_t s) {
  const int tokens = TILES ? (d.pos.per_seq + CH - 1) / CH * CH : d.pos.per_seq;
  const dim3 grid((tokens + PREP_TOKENS - 1) / PREP_TOKENS, (2 * d.kv_heads + d.heads + 3) / 4, d.rows / d.pos.per_seq);
  auto k = !d.conv ? prepare_kernel<T, TZ, -1, TILES> : d.taps <= 4 ? prepare_kernel<T, TZ, 4, TILES> : prepare_kernel<T, TZ, 0, TILES>;
  k<<<grid, 128, 0, s>>>(d, (T*)out, norms, beta_g);
  return cudaGetLastError();
}
cudaError_t launch_prepare(const DeltaInputs& d, bool tiles, void* out, float* norms, float* beta_g, cudaStream_t s) {
  if (tiles && (d.f32 || !recurrence_chunks_supported(d.dp))) return cudaErrorInvalidValue;
  if (d.f32 != d.z_f32) return cudaErrorInvalidValue;
  if (d.f32) return launch_prepare<float, float, false>(d, out, norms, beta_g, s);
  return tiles ? launch_prepare<bf16, bf16, true>(d, out, norms, beta_g, s) : launch_prepare<bf16, bf16, false>(d, out, norms, beta_g, s);
}

}  // namespace

cudaError_t delta_prepare(const DeltaInputs& d, bool tiles, void* out, float* norms, float* beta_g, cudaStream_t s) {
  if (!inputs_ok(d) || !d.ba || !norms || !beta_g) return cudaErrorInvalidValue;
  return launch_prepare(d, tiles, out, norms, beta_g, s);
}

cudaError_t decay_prepare(bool f32, const void* z, long long ldz, int rows, int per_seq, int heads, int dp, int vp, bool tiles, void* out, cudaStream_t s) {
  DeltaInputs d{};
  d.f32 = d.z_f32 = f32; d.z = z; d.ldz = ldz; d.rows = rows; d.heads = d.kv_heads = heads; d.dp = dp; d.vp = vp; d.taps = 1;
  d.pos.per_seq = per_seq;
  if (!sizes_ok(d)) return cudaErrorInvalidValue;
  return launch_prepare(d, tiles, out, nullptr, nullptr, s);
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
size_t recurrence_tiles(int seqs, int per_seq, int heads, int kv_heads, int dp, int vp) {
  return (size_t)Tiles(seqs, per_seq, heads, kv_heads, dp, vp).elements(seqs, heads) * 2;
}
size_t recurrence_scratch(int seqs, int per_seq, int heads, bool delta) {
  return (size_t)seqs * ((per_seq + CH - 1) / CH) * heads * chunk_bytes(delta);
}

template <bool DELTA, int D>
static cudaError_t launch_chunks(const Recurrence& d, uint8_t* scratch, int* status, cudaStream_t s) {
  static PerDeviceOnce configured;
  constexpr int SMEM = ScanSmem<DELTA, D>::TOTAL;
  cudaError_t e = configured.once([] { return cudaFuncSetAttribute(chunk_scan_kernel<DELTA, D>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM); });
  if (e != cudaSuccess) return e;
  const int seqs = d.rows / d.pos.per_seq, chunks = (d.pos.per_seq + CH - 1) / CH;
  chunk_gram_kernel<DELTA, D><<<dim3(chunks, d.heads, seqs), 256, 0, s>>>(d, scratch);
  e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  chunk_scan_kernel<DELTA, D><<<dim3((d.vp + VS - 1) / VS, d.heads, seqs), SCAN_THREADS, SMEM, s>>>(d, scratch, status);
  return cudaGetLastError();
}
cudaError_t recurrence_chunks(const Recurrence& d, void* scratch, int* status, cudaStream_t s) {
  if (!recurrence_ok(d) || d.f32 || !recurrence_chunks_supported(d.dp) || !scratch) return cudaErrorInvalidValue;
  uint8_t* p = (uint8_t*)scratch;
  if (tile_dim(d.dp) == 64) return d.beta_g ? launch_chunks<true, 64>(d, p, status, s) : launch_chunks<false, 64>(d, p, status, s);
  return d.beta_g ? launch_chunks<true, 128>(d, p, status, s) : launch_chunks<false, 128>(d, p, status, s);
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
  const int lanes = np <= 64 ? 8 : np <= 128 ? 16 : 32;
  const int blocks = (int)(((long long)rows * groups * lanes + 255) / 256);
  const int extra = ring ? (ring->taps - 1) * (ring->rows / ring->pos.per_seq) : 0;
  const DeltaInputs in = ring ? *ring : DeltaInputs{};
  auto go = [&](auto k8, auto k16, auto k32) {
    (lanes == 8 ? k8 : lanes == 16 ? k16 : k32)<<<blocks + extra, 256, 0, s>>>(d, in, blocks);
    return cudaGetLastError();
  };
  if (f32) return go(norm_gate_warp_kernel<float, 8>, norm_gate_warp_kernel<float, 16>, norm_gate_warp_kernel<float, 32>);
  return go(norm_gate_warp_kernel<bf16, 8>, norm_gate_warp_kernel<bf16, 16>, norm_gate_warp_kernel<bf16, 32>);
}

}  // namespace serve
}  // namespace nc
