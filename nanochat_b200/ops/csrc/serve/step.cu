// One token per row through the mixers of recurrent.cu and window.cu, from the projections to what the output product
// reads.
//
//   delta_step      a CTA per (head, row): convolution, unit norms, step size and decay, state, norm and gate
//   parallel_step   window attention and fixed-decay heads side by side in one grid of clusters
//       attention   a cluster per (16 query heads of a key head, row) splits the window's keys; the CTA that covers the
//                   newest key takes it from the projection and appends it to the store; the partial results meet in
//                   distributed shared memory
//       decay       a CTA per (head, row) updates its state; the row's last CTA to finish norms and gates the row
//
// What the step before has left (states, convolution inputs, stored keys, lengths) and the weights are read before the wait on
// the kernel in front, the layer's input product. Both recurrences read out what they write without a second pass over the
// state: (g S + k u^T)^T q = g S^T q + (k . q) u.
#include <cooperative_groups.h>

#include "mma.cuh"

namespace nc {
namespace serve {

namespace {

namespace cg = cooperative_groups;

constexpr int THREADS = 256;
constexpr int MAX_NR = 32;               // state rows a thread holds, four columns each

template <typename T> __device__ __forceinline__ float silu_of(float v) { return v * sigmoid_of<T>(v); }
template <typename TZ> __device__ __forceinline__ float zf(const void* z, long long i) { return to_f(((const TZ*)z)[i]); }

// A state of dp x vp floats over the block: thread (column group vi, row group grp) holds NR neighbouring rows, from grp * NR
// on, of four columns. dp is a multiple of 8, NR of 4: rows come and go in fours.
template <int NR>
struct StateTile {
  float s[NR][4];
  int vi, grp, d0, groups;
  bool on;
  __device__ void load(const float* st, int dp, int vp) {
    const int vt = vp / 4;
    groups = (dp + NR - 1) / NR;
    vi = threadIdx.x % vt;
    grp = threadIdx.x / vt;
    d0 = grp * NR;
    on = grp < groups;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const float4 v = d0 + i < dp ? *reinterpret_cast<const float4*>(st + (long long)(d0 + i) * vp + vi * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[i][0] = v.x; s[i][1] = v.y; s[i][2] = v.z; s[i][3] = v.w;
    }
  }
  __device__ void clear() {
#pragma unroll
    for (int i = 0; i < NR; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
  }
  __device__ static void four(const float* x, int d, int dp, float (&f)[4]) {
    const float4 v = d < dp ? *reinterpret_cast<const float4*>(x + d) : make_float4(0.f, 0.f, 0.f, 0.f);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
  // this thread's part of S^T x, left in part[grp][columns]; with y, returns the row group's part of x . y
  __device__ float dot(const float* x, int dp, int vp, float* part, const float* y = nullptr) const {
    float p[4] = {0.f, 0.f, 0.f, 0.f}, xy = 0.f;
#pragma unroll
    for (int i = 0; i < NR; i += 4) {
      float xv[4], yv[4];
      four(x, d0 + i, dp, xv);
      if (y) four(y, d0 + i, dp, yv);
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        if (y) xy += xv[r] * yv[r];
#pragma unroll
        for (int j = 0; j < 4; ++j) p[j] += s[i + r][j] * xv[r];
      }
    }
    if (on) *reinterpret_cast<float4*>(part + grp * vp + vi * 4) = make_float4(p[0], p[1], p[2], p[3]);
    return xy;
  }
  // S <- g S + k u^T
  __device__ void update(float g, const float* k, const float (&u)[4], int dp) {
#pragma unroll
    for (int i = 0; i < NR; i += 4) {
      float kv[4];
      four(k, d0 + i, dp, kv);
#pragma unroll
      for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int j = 0; j < 4; ++j) s[i + r][j] = g * s[i + r][j] + kv[r] * u[j];
    }
  }
  __device__ void store(float* st, int dp, int vp) const {
#pragma unroll
    for (int i = 0; i < NR; ++i)
      if (d0 + i < dp) *reinterpret_cast<float4*>(st + (long long)(d0 + i) * vp + vi * 4) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
  }
};
__device__ __forceinline__ void sum_parts(const float* part, int groups, int vp, int col, float (&t)[4]) {
  t[0] = t[1] = t[2] = t[3] = 0.f;
#pragma unroll 8
  for (int g = 0; g < groups; ++g) {
    const float4 a = *reinterpret_cast<const float4*>(part + g * vp + col);
    t[0] += a.x; t[1] += a.y; t[2] += a.z; t[3] += a.w;
  }
}
// floats of dynamic shared memory: q, k (dp), v (vp), two partial sums of up to THREADS * 4 each, the row groups' k . q
__host__ __device__ constexpr int step_floats(int dp, int vp) { return 2 * dp + vp + 2 * THREADS * 4 + THREADS; }
constexpr int MAX_CHANNELS = 6 * THREADS;      // q, k and v of one head

template <typename T, typename TZ, int NR>
__global__ void __launch_bounds__(THREADS)
delta_step_kernel(const DeltaStep d) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[2][32];
  __shared__ float s_beta, s_g;
  constexpr int PER = MAX_CHANNELS / THREADS;
  const DeltaInputs& in = d.in;
  const int h = blockIdx.x, row = blockIdx.y, rep = in.heads / in.kv_heads, kvh = h / rep;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dp = in.dp, vp = in.vp, channels = 2 * in.kv_heads * dp + in.heads * vp, mine = 2 * dp + vp;
  float *sq = sm, *sk = sm + dp, *sv = sm + 2 * dp, *part_k = sv + vp, *part_q = part_k + THREADS * 4, *part_kq = part_q + THREADS * 4;
  float* state = d.state.ptr + row * d.state.seq_stride + (long long)h * dp * vp;
  float* ring = in.ring.ptr + row * in.ring.seq_stride;
  const int pos = in.pos.lens[row], slot = pos % in.taps;
  StateTile<NR> S;
  S.load(state, dp, vp);
  auto channel = [&](int c) { return c < dp ? kvh * dp + c : c < 2 * dp ? in.kv_heads * dp + kvh * dp + c - dp : 2 * in.kv_heads * dp + h * vp + c - 2 * dp; };
  float past[PER], w_now[PER];                     // the convolution without the current token, and its weight
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int c = tid + i * THREADS;
    past[i] = w_now[i] = 0.f;
    if (c < mine) {
      const int ch = channel(c);
      w_now[i] = in.conv[(long long)(in.taps - 1) * channels + ch];
      for (int t = 1; t < in.taps && t <= pos; ++t) {
        const int at = slot - t < 0 ? slot - t + in.taps : slot - t;
        past[i] += in.conv[(long long)(in.taps - 1 - t) * channels + ch] * ring[(long long)at * channels + ch];
      }
    }
  }
  const float bias = in.dt_bias[h], neg_a = in.neg_a[h];
  if (pos == 0) S.clear();
  const int col = S.vi * 4;
  float norm[4], gate[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) norm[j] = S.grp == 0 ? d.norm[col + j] : 0.f;
  pdl_wait();
  pdl_trigger();
  float x[PER], beta_in = 0.f, decay_in = 0.f;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int c = tid + i * THREADS;
    x[i] = c < mine ? zf<TZ>(in.z, row * in.ldz + channel(c)) : 0.f;
  }
  if (tid == THREADS - 1) {
    beta_in = in.ba[row * in.ldba + h];
    decay_in = in.ba[row * in.ldba + in.a_off + h] + bias;
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) gate[j] = S.grp == 0 ? zf<TZ>(in.z, row * in.ldz + d.gate_off + (long long)h * vp + col + j) : 0.f;
  float ss[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int c = tid + i * THREADS;
    if (c >= mine) continue;
    const float a = silu_of<T>(past[i] + w_now[i] * x[i]);
    sm[c] = a;
    if (c < 2 * dp) ss[c >= dp] += a * a;
    if (c >= 2 * dp || h % rep == 0) ring[(long long)slot * channels + channel(c)] = x[i];      // one writer per channel
  }
  if (tid == THREADS - 1) {
    s_beta = sigmoidf(beta_in);
    s_g = expf(neg_a * (decay_in > 20.f ? decay_in : log1pf(expf(decay_in))));
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    ss[i] = warp_sum(ss[i]);
    if (lane == 0) red[i][warp] = ss[i];
  }
  __syncthreads();
  S.dot(sk, dp, vp, part_k);
  const float kq_part = S.dot(sq, dp, vp, part_q, sk);
  if (S.on && S.vi == 0) part_kq[S.grp] = kq_part;
  ss[0] = ss[1] = 0.f;
#pragma unroll
  for (int w = 0; w < THREADS / 32; ++w) { ss[0] += red[0][w]; ss[1] += red[1][w]; }
  const float rq = 1.f / sqrtf((ss[0] + 1e-6f) * in.dim), rk = 1.f / sqrtf(ss[1] + 1e-6f), g = s_g;
  __syncthreads();
  float u[4] = {0.f, 0.f, 0.f, 0.f}, o[4] = {0.f, 0.f, 0.f, 0.f}, so[1] = {0.f};
  if (S.on) {
    float t[4];
    sum_parts(part_k, S.groups, vp, col, t);
#pragma unroll
    for (int j = 0; j < 4; ++j) u[j] = rk * s_beta * (sv[col + j] - g * rk * t[j]);
  }
  if (S.grp == 0) {                                // the first threads read out
    float t[4], kq = 0.f;
    sum_parts(part_q, S.groups, vp, col, t);
#pragma unroll 8
    for (int i = 0; i < S.groups; ++i) kq += part_kq[i];
#pragma unroll
    for (int j = 0; j < 4; ++j) { o[j] = rq * (g * t[j] + kq * u[j]); so[0] += o[j] * o[j]; }
  }
  if (vp <= 128) so[0] = warp_sum(so[0]);          // they are lanes of one warp
  else block_sum<1>(so, red[0]);
  if (S.grp == 0) {
    const float r = inv_rms(so[0], in.vdim, d.eps);
#pragma unroll
    for (int j = 0; j < 4; ++j) ((T*)d.y)[row * d.ldy + (long long)h * vp + col + j] = from_f<T>(o[j] * r * norm[j] * silu_of<T>(gate[j]));
  }
  S.update(g, sk, u, dp);
  S.store(state, dp, vp);
}

// ------------------------------------------------------------------------- fixed decay
template <typename T, typename TZ, int NR>
__device__ void decay_head(const DecayStep& d, int h, int row, float* sm) {
  __shared__ float red[32];
  __shared__ int s_last;
  const int tid = threadIdx.x, dp = d.dp, vp = d.vp, width = d.heads * vp;
  float *sq = sm, *sk = sm + dp, *sv = sm + 2 * dp, *part = sv + vp, *part_kq = part + 2 * THREADS * 4;
  float* state = d.state.ptr + row * d.state.seq_stride + (long long)h * dp * vp;
  StateTile<NR> S;
  S.load(state, dp, vp);
  if (d.pos.lens[row] == 0) S.clear();
  const float g = expf(d.log_decay[h]);
  pdl_wait();
  pdl_trigger();
  for (int c = tid; c < 2 * dp + vp; c += THREADS) {
    const int at = c < dp ? d.q_off + h * dp + c : c < 2 * dp ? d.k_off + h * dp + c - dp : d.v_off + h * vp + c - 2 * dp;
    sm[c] = silu_of<T>(zf<TZ>(d.z, row * d.ldz + at));
  }
  __syncthreads();
  const float kq_part = S.dot(sq, dp, vp, part, sk);
  if (S.on && S.vi == 0) part_kq[S.grp] = kq_part;
  __syncthreads();
  float* o = d.o + (long long)row * width;
  const int col = S.vi * 4;
  if (S.grp == 0) {
    float t[4], kq = 0.f;
    sum_parts(part, S.groups, vp, col, t);
#pragma unroll 8
    for (int i = 0; i < S.groups; ++i) kq += part_kq[i];
    *reinterpret_cast<float4*>(o + h * vp + col) =
        make_float4(g * t[0] + kq * sv[col], g * t[1] + kq * sv[col + 1], g * t[2] + kq * sv[col + 2], g * t[3] + kq * sv[col + 3]);
    __threadfence();
  }
  __syncthreads();
  if (tid == 0) s_last = atomicAdd(d.done + row, 1) == d.heads - 1;
  if (S.on) {
    const float u[4] = {sv[col], sv[col + 1], sv[col + 2], sv[col + 3]};
    S.update(g, sk, u, dp);
    S.store(state, dp, vp);
  }
  __syncthreads();
  if (!s_last) return;
  if (tid == 0) d.done[row] = 0;
  __threadfence();
  float ss[1] = {0.f};
  for (int c = tid * 4; c < width; c += THREADS * 4) {
    const float4 v = __ldcg(reinterpret_cast<const float4*>(o + c));
    ss[0] += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  block_sum<1>(ss, red);
  const float r = inv_rms(ss[0], d.heads * d.vdim, d.eps) * d.out_scale;
  for (int c = tid; c < width; c += THREADS)
    ((T*)d.y)[row * d.ldy + c] = from_f<T>(__ldcg(o + c) * r * d.norm[c] * sigmoid_of<T>(zf<TZ>(d.z, row * d.ldz + d.gate_off + c)));
}

// --------------------------------------------------------------------------- attention
constexpr int KT = 64;                       // keys per tile
constexpr int AW = THREADS / 32;
__host__ __device__ constexpr int padded(int dp) { return (dp + 31) / 32 * 32; }           // scores step through 32 columns
__host__ __device__ constexpr size_t window_smem(int dp) {
  return (size_t)(16 + 2 * KT) * (padded(dp) + 8) * 2 + (size_t)16 * (KT + 8) * 2 + (size_t)16 * padded(dp) * 4 + (size_t)padded(dp) * 4;
}

// NU: 16-column units of the values per warp (dp <= 128 * NU). All CTAs of the cluster call this with their rank as `split`.
template <typename TZ, int NU>
__device__ void window_group(const WindowAttn& d, int group, int row, uint8_t* smem, int* status) {
  cg::cluster_group cluster = cg::this_cluster();
  const int split = cluster.block_rank(), splits = cluster.num_blocks();
  __shared__ float s_max[AW][16], s_sum[AW][16], s_m[16], s_l[16];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rep = d.heads / d.kv_heads, tiles = (rep + 15) / 16, kvh = group / tiles, part = group - kvh * tiles;
  const int h0 = kvh * rep + part * 16, heads = min(16, rep - part * 16);
  const int DP = padded(d.dp), LD = DP + 8, LP = KT + 8, nk = d.kv_heads * d.dp;
  bf16* sQ = reinterpret_cast<bf16*>(smem);
  bf16* sK = sQ + 16 * LD;
  bf16* sV = sK + KT * LD;
  bf16* sP = sV + KT * LD;
  float* sO = reinterpret_cast<float*>(sP + 16 * LP);                // 16 x DP
  float2* s_cs = reinterpret_cast<float2*>(sO + 16 * DP);
  for (int i = tid; i < (16 + 2 * KT) * ((DP - d.dp) / 8); i += THREADS) {      // columns that only fill up a step
    const int per = (DP - d.dp) / 8, r = i / per;
    *reinterpret_cast<uint4*>(sQ + r * LD + d.dp + (i - r * per) * 8) = make_uint4(0, 0, 0, 0);
  }
  const int pos = d.pos.lens[row];
  const KeyRange kr = split_keys(pos, d.window, splits, split, KT);
  const bool any = kr.begin < kr.end;
  auto load_tile = [&](int tile) {                                   // the newest key comes from the projection instead
    const int mine = tile + warp * 8 + (lane & 7);
    const long long my_off = mine < kr.end && mine < pos ? token_offset(d.pg, row, mine) : -1;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const long long off = __shfl_sync(0xffffffffu, my_off, k);
      const int r = warp * 8 + k;
      if (tile + r == pos) continue;
      const bf16* src = (const bf16*)d.pg.pool + (off >= 0 ? off + kvh * d.dp : 0);
      for (int c = lane * 8; c < d.dp; c += 256) {
        cp_async16_or_zero(sK + r * LD + c, src + c, off >= 0);
        cp_async16_or_zero(sV + r * LD + c, src + (off >= 0 ? nk : 0) + c, off >= 0);
      }
    }
    cp_async_commit();
  };
  float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.f, 0.f};
  float o[NU][2][4];
#pragma unroll
  for (int u = 0; u < NU; ++u)
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[u][t][e] = 0.f;
  const int units = DP / 16;
  if (any) {
    load_tile(kr.begin);
    for (int i = tid; i < d.dims / 2; i += THREADS) s_cs[i] = turn_of(pos, d.freq, i, d.dims / 2);
  }
  pdl_wait();
  pdl_trigger();
  if (any) {
    __syncthreads();
    const TZ* z = (const TZ*)d.z + row * d.ldz;
    const int pairs = d.dp / 2;
    for (int i = tid; i < 16 * pairs; i += THREADS) {
      const int h = i / pairs, c = (i - h * pairs) * 2;
      float a = 0.f, b = 0.f;
      if (h < heads) {
        a = to_f(z[d.q_off + (long long)(h0 + h) * d.dp + c]);
        b = to_f(z[d.q_off + (long long)(h0 + h) * d.dp + c + 1]);
        if (c < d.dims) {
          const float2 t = s_cs[c >> 1];
          const float u = a * t.x - b * t.y;
          b = b * t.x + a * t.y;
          a = u;
        }
      }
      *reinterpret_cast<uint32_t*>(sQ + h * LD + c) = pack_bf16(a, b);
    }
    const float sc = d.scale * 1.4426950408889634f, cap = d.softcap * 1.4426950408889634f;
    for (int tile = kr.begin; tile < kr.end; tile += KT) {
      if (pos >= tile && pos < tile + KT) {                          // the newest key: into its place and into the store
        const int r = pos - tile;
        const long long off = token_offset(d.pg, row, pos);
        if (off < 0 && tid == 0 && part == 0 && status) atomicCAS(status, 0, (ST_BAD_ARG << 24) | 0x57044);   // no page: not stored
        bf16* entry = off >= 0 && part == 0 ? (bf16*)d.pg.pool + off + kvh * d.dp : nullptr;
        for (int i = tid; i < pairs; i += THREADS) {
          const int c = i * 2;
          const float a = to_f(z[d.k_off + kvh * d.dp + c]), b = to_f(z[d.k_off + kvh * d.dp + c + 1]);
          const float2 t = c < d.dims ? s_cs[i] : make_float2(1.f, 0.f);
          const uint32_t turned = pack_bf16(a * t.x - b * t.y, b * t.x + a * t.y), plain = pack_bf16(a, b);
          *reinterpret_cast<uint32_t*>(sK + r * LD + c) = turned;
          *reinterpret_cast<uint32_t*>(sV + r * LD + c) = plain;
          if (entry) {
            *reinterpret_cast<uint32_t*>(entry + c) = turned;
            *reinterpret_cast<uint32_t*>(entry + nk + c) = plain;
          }
        }
      }
      cp_async_wait<0>();
      __syncthreads();
      float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      const bf16* qp = sQ + (lane & 15) * LD + (lane >> 4) * 8;
      const bf16* kp = sK + (warp * 8 + (lane & 7)) * LD + (lane >> 3) * 8;
#pragma unroll 4
      for (int k = 0; k < DP; k += 32) {
        uint32_t a0[4], a1[4], b[4];
        ldmatrix4(a0, qp + k);
        ldmatrix4(a1, qp + k + 16);
        ldmatrix4(b, kp + k);
        mma_16816(s[0], a0, b[0], b[1]);
        mma_16816(s[1], a1, b[2], b[3]);
      }
      const int j = tile + warp * 8 + (lane & 3) * 2;
      float mx[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float v = s[0][r * 2 + e] + s[1][r * 2 + e];
          v = d.softcap > 0.f ? cap * tanhf(v * d.scale / d.softcap) : v * sc;
          s[0][r * 2 + e] = j + e < kr.end ? v : NEG_BIG;
        }
        mx[r] = fmaxf(s[0][r * 2], s[0][r * 2 + 1]);
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        if ((lane & 3) == 0) s_max[warp][(lane >> 2) + r * 8] = mx[r];
      }
      __syncthreads();
      float alpha[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int hr = (lane >> 2) + r * 8;
        float m_new = m_run[r];
#pragma unroll
        for (int w = 0; w < AW; ++w) m_new = fmaxf(m_new, s_max[w][hr]);
        alpha[r] = exp2f(m_run[r] - m_new);
        m_run[r] = m_new;
        const float p0 = j < kr.end ? exp2f(s[0][r * 2] - m_new) : 0.f;
        const float p1 = j + 1 < kr.end ? exp2f(s[0][r * 2 + 1] - m_new) : 0.f;
        l_run[r] = l_run[r] * alpha[r] + p0 + p1;
        *reinterpret_cast<uint32_t*>(sP + hr * LP + warp * 8 + (lane & 3) * 2) = pack_bf16(p0, p1);
      }
      __syncthreads();
#pragma unroll
      for (int u = 0; u < NU; ++u)
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) o[u][t][e] *= alpha[e >> 1];
#pragma unroll
      for (int k = 0; k < KT; k += 16) {
        uint32_t a[4];
        ldmatrix4(a, sP + (lane & 15) * LP + k + (lane >> 4) * 8);
#pragma unroll
        for (int u = 0; u < NU; ++u) {
          const int unit = warp + u * AW;
          if (unit < units) {
            uint32_t b[4];
            ldmatrix4_trans(b, sV + (k + (lane & 15)) * LD + unit * 16 + (lane >> 4) * 8);
            mma_16816(o[u][0], a, b[0], b[1]);
            mma_16816(o[u][1], a, b[2], b[3]);
          }
        }
      }
      if (tile + KT < kr.end) {
        __syncthreads();                                             // the tile has been read
        load_tile(tile + KT);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    const int h = (lane >> 2) + r * 8;
    if ((lane & 3) == 0) s_sum[warp][h] = l_run[r];
    if (warp == 0 && (lane & 3) == 0) s_m[h] = m_run[r];
#pragma unroll
    for (int u = 0; u < NU; ++u) {
      const int unit = warp + u * AW;
      if (unit >= units) continue;
#pragma unroll
      for (int t = 0; t < 2; ++t)
        *reinterpret_cast<float2*>(sO + h * DP + unit * 16 + t * 8 + (lane & 3) * 2) = make_float2(o[u][t][r * 2], o[u][t][r * 2 + 1]);
    }
  }
  __syncthreads();
  if (tid < 16) {
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < AW; ++w) l += s_sum[w][tid];
    s_l[tid] = l;
  }
  cluster.sync();
  for (int h = split; h < heads; h += splits) {                      // every CTA closes some of the heads
    float M = NEG_BIG, L = 0.f;
    for (int r = 0; r < splits; ++r) M = fmaxf(M, *cluster.map_shared_rank(&s_m[h], r));
    for (int r = 0; r < splits; ++r) L += *cluster.map_shared_rank(&s_l[h], r) * exp2f(*cluster.map_shared_rank(&s_m[h], r) - M);
    const float f = L > 0.f ? d.out_scale / L : 0.f;
    bf16* y = (bf16*)d.y + row * d.ldy + (long long)(h0 + h) * d.dp;
    for (int c = tid; c < d.dp; c += THREADS) {
      float v = 0.f;
      for (int r = 0; r < splits; ++r)
        v += cluster.map_shared_rank(sO, r)[h * DP + c] * exp2f(*cluster.map_shared_rank(&s_m[h], r) - M);
      y[c] = __float2bfloat16_rn(v * f);
    }
  }
  cluster.sync();                                                    // the others' shared memory stays until it has been read
}

// grid (cluster, key groups + ceil(decay heads / cluster), rows)
template <typename T, typename TZ, int NU, int NR>
__global__ void __launch_bounds__(THREADS)
parallel_step_kernel(const WindowAttn left, const DecayStep right, int groups, int* status) {
  extern __shared__ __align__(16) uint8_t smem[];
  if constexpr (NU > 0) {
    if ((int)blockIdx.y < groups) {
      window_group<TZ, NU>(left, blockIdx.y, blockIdx.z, smem, status);
      return;
    }
  }
  if constexpr (NR > 0) {
    const int h = ((int)blockIdx.y - groups) * gridDim.x + blockIdx.x;
    if (h < right.heads) {
      decay_head<T, TZ, NR>(right, h, blockIdx.z, reinterpret_cast<float*>(smem));
      return;
    }
  }
  pdl_wait();                              // a CTA that only fills up the grid must not let the kernel end early
  pdl_trigger();
}

int state_rows(int dp, int vp) {           // state rows per thread, 0: the state does not fit the block
  if (vp <= 0 || (vp & 3) || vp / 4 > THREADS || dp <= 0) return 0;
  const int groups = THREADS / (vp / 4), n = (dp + groups - 1) / groups;
  return n <= 4 ? 4 : n <= 8 ? 8 : n <= 16 ? 16 : n <= MAX_NR ? MAX_NR : 0;
}

template <typename T, typename TZ>
cudaError_t launch_delta(const DeltaStep& d, cudaStream_t s) {
  const dim3 grid(d.in.heads, d.in.rows);
  const size_t smem = step_floats(d.in.dp, d.in.vp) * sizeof(float);
  switch (state_rows(d.in.dp, d.in.vp)) {
    case 4: return launch_pdl(delta_step_kernel<T, TZ, 4>, grid, dim3(THREADS), smem, s, d);
    case 8: return launch_pdl(delta_step_kernel<T, TZ, 8>, grid, dim3(THREADS), smem, s, d);
    case 16: return launch_pdl(delta_step_kernel<T, TZ, 16>, grid, dim3(THREADS), smem, s, d);
    case 32: return launch_pdl(delta_step_kernel<T, TZ, 32>, grid, dim3(THREADS), smem, s, d);
  }
  return cudaErrorInvalidValue;
}

template <typename T, typename TZ, int NU, int NR>
cudaError_t launch_parallel(const WindowAttn& left, const DecayStep& right, int* status, cudaStream_t s) {
  static PerDeviceOnce configured;
  auto kern = parallel_step_kernel<T, TZ, NU, NR>;
  const cudaError_t e = configured.once([&] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024); });
  if (e != cudaSuccess) return e;
  size_t smem = NR > 0 ? step_floats(right.dp, right.vp) * sizeof(float) : 0;
  int splits = 1, groups = 0;
  if (NU > 0) {
    if (window_smem(left.dp) > smem) smem = window_smem(left.dp);
    const int keys = left.window > 0 ? left.window : left.pg.max_pages << left.pg.shift;
    while (splits < 8 && splits * KT < keys) splits *= 2;
    const int rep = left.heads / left.kv_heads;
    groups = left.kv_heads * ((rep + 15) / 16);
  }
  if (smem > 160 * 1024) return cudaErrorInvalidValue;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(splits, groups + (NR > 0 ? (right.heads + splits - 1) / splits : 0), NU > 0 ? left.rows : right.rows);
  cfg.blockDim = dim3(THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute at[2];
  at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  at[0].val.programmaticStreamSerializationAllowed = 1;
  at[1].id = cudaLaunchAttributeClusterDimension;
  at[1].val.clusterDim.x = splits; at[1].val.clusterDim.y = 1; at[1].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 2;
  return cudaLaunchKernelEx(&cfg, kern, left, right, groups, status);
}

template <typename T, typename TZ, int NU>
cudaError_t launch_parallel_rows(const WindowAttn& left, const DecayStep& right, int nr, int* status, cudaStream_t s) {
  switch (nr) {
    case 0: if constexpr (NU > 0) return launch_parallel<T, TZ, NU, 0>(left, right, status, s); else return cudaErrorInvalidValue;
    case 4: return launch_parallel<T, TZ, NU, 4>(left, right, status, s);
    case 8: return launch_parallel<T, TZ, NU, 8>(left, right, status, s);
    case 16: return launch_parallel<T, TZ, NU, 16>(left, right, status, s);
    case 32: return launch_parallel<T, TZ, NU, 32>(left, right, status, s);
  }
  return cudaErrorInvalidValue;
}

}  // namespace

bool delta_step_supported(int dp, int vp) { return !(dp & 7) && !(vp & 7) && state_rows(dp, vp) > 0 && 2 * dp + vp <= MAX_CHANNELS; }
bool decay_step_supported(int dp, int vp) { return delta_step_supported(dp, vp); }
bool window_step_supported(bool f32, int dp) { return !f32 && dp > 0 && dp <= 256 && !(dp & 7); }

cudaError_t delta_step(const DeltaStep& d, cudaStream_t s) {
  const DeltaInputs& in = d.in;
  if (in.rows <= 0 || in.rows > 65535 || in.heads > 65535 || in.pos.per_seq != 1 || !in.pos.lens || in.heads <= 0 || in.kv_heads <= 0 || in.heads % in.kv_heads || in.taps <= 0 ||
      !delta_step_supported(in.dp, in.vp) || in.dim > in.dp || in.vdim > in.vp || !in.z || !in.ba || !in.ring.ptr || !d.state.ptr || (d.state.seq_stride & 3) ||
      !d.y || (in.f32 && !in.z_f32))
    return cudaErrorInvalidValue;
  if (in.f32) return launch_delta<float, float>(d, s);
  return in.z_f32 ? launch_delta<bf16, float>(d, s) : launch_delta<bf16, bf16>(d, s);
}

cudaError_t parallel_step(const WindowAttn* left, const DecayStep* right, int* status, cudaStream_t s) {
  if (!left && !right) return cudaErrorInvalidValue;
  int nu = 0, nr = 0;
  bool f32 = false, z_f32 = false;
  if (left) {
    const Pages& p = left->pg;
    if (!window_step_supported(left->f32, left->dp) || left->rows <= 0 || left->rows > 65535 || left->pos.per_seq != 1 || !left->pos.lens || left->heads <= 0 ||
        left->kv_heads <= 0 || left->heads % left->kv_heads || left->dims < 0 || left->dims > left->dp || (left->dims & 1) || !left->z || !left->y || !p.pool ||
        !p.table || p.max_pages <= 0 || p.shift < 0 || p.shift > 16 || p.n_pages <= 0 || p.width != 2 * left->kv_heads * left->dp)
      return cudaErrorInvalidValue;
    nu = left->dp <= 128 ? 1 : 2;
    z_f32 = left->z_f32;
  }
  if (right) {
    nr = state_rows(right->dp, right->vp);
    if (!decay_step_supported(right->dp, right->vp) || right->rows <= 0 || right->rows > 65535 || right->pos.per_seq != 1 || !right->pos.lens || right->heads <= 0 ||
        right->vdim > right->vp || !right->z || !right->log_decay || !right->state.ptr || (right->state.seq_stride & 3) || !right->norm || !right->o ||
        !right->done || !right->y || (right->f32 && !right->z_f32))
      return cudaErrorInvalidValue;
    f32 = right->f32;
    if (left && (right->rows != left->rows || right->z_f32 != z_f32 || f32)) return cudaErrorInvalidValue;
    z_f32 = right->z_f32;
  }
  const WindowAttn l = left ? *left : WindowAttn{};
  const DecayStep r = right ? *right : DecayStep{};
  if (f32) return launch_parallel_rows<float, float, 0>(l, r, nr, status, s);
  if (nu == 0) return z_f32 ? launch_parallel_rows<bf16, float, 0>(l, r, nr, status, s) : launch_parallel_rows<bf16, bf16, 0>(l, r, nr, status, s);
  if (nu == 1) return z_f32 ? launch_parallel_rows<bf16, float, 1>(l, r, nr, status, s) : launch_parallel_rows<bf16, bf16, 1>(l, r, nr, status, s);
  return z_f32 ? launch_parallel_rows<bf16, float, 2>(l, r, nr, status, s) : launch_parallel_rows<bf16, bf16, 2>(l, r, nr, status, s);
}

}  // namespace serve
}  // namespace nc
