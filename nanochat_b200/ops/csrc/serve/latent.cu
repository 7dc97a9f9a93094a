// Latent attention over a paged store of [normed latent | rotated shared key part] entries.
//
//   latent_post      query latent norm, the step's entries into the store (and a dense copy for whole prompts)
//   latent_gather    stored entries of a token range as dense rows (keys a prompt portion sees from before it)
//   rotate_heads     rotary turn of every head's rotated query part, in place
//   absorb_query     q_h Wuk_h: with the key projection moved to the query side, scores are dot products with entries
//   latent_attention absorbed queries against the stored entries of a key range, split over CTAs; every split leaves
//                    an unnormalised partial. bf16: one CTA serves 16 heads of a row, so an entry is fetched once for
//                    all of them, and both products run on mma.sync with the latents staged in shared memory by
//                    cp.async. Otherwise (float, or entries too wide for shared memory): a CTA per head, plain dots.
//   latent_values    combines the splits and applies the value projection
// Scores and weights are float; the exponent base is 2 (scale carries log2 e).
#include "latent_store.cuh"
#include "mma.cuh"

namespace nc {
namespace serve {

namespace {

constexpr int MAX_SPLITS = 32;

// ---------------------------------------------------------------------- post / gather
// grid (rows, 1 or 2): y = 0 the store entry, y = 1 the query latent. The norm weights' padding is zero.
template <typename T, typename TZ>
__global__ void __launch_bounds__(128)
latent_post_kernel(const LatentPost d, int* status) {
  __shared__ float red[32];
  const int row = blockIdx.x;
  const TZ* z = (const TZ*)d.z + (long long)row * d.ldz;
  if (blockIdx.y == 1) {
    float ss[1] = {0.f};
    for (int c = threadIdx.x * 8; c < d.qp; c += 1024) {
      float v[8];
      load8(z + c, v);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss[0] += v[j] * v[j];
    }
    block_sum<1>(ss, red);
    const float r = inv_rms(ss[0], d.q_rank, d.eps);
    T* cq = (T*)d.cq + (long long)row * d.ldcq;
    for (int c = threadIdx.x * 8; c < d.qp; c += 1024) {
      float v[8], w[8];
      load8(z + c, v);
      load8(d.q_w + c, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] *= r * w[j];
      store8(cq + c, v);
    }
    return;
  }
  int seq;
  const int pos = row_position(d.pos, row, seq);
  const long long off = token_offset(d.pg, seq, pos);
  if (off < 0 && threadIdx.x == 0 && status) atomicCAS(status, 0, (ST_BAD_ARG << 24) | 0x57043);   // no page: not stored
  store_latent<T, TZ>(z + d.c_off, z + d.rot_off, d.kv_rank, d.kvp, d.kv_w, d.eps, d.rot_dim, d.rp, d.dims, d.freq, pos,
                      off < 0 ? nullptr : (T*)d.pg.pool + off,
                      d.kv_out ? (T*)d.kv_out + (long long)row * d.ldkv : nullptr, red);
}

template <typename T>
__global__ void __launch_bounds__(128)
latent_gather_kernel(const Pages pg, int seq, int first, T* out, long long ldo, int* status) {
  const int j = blockIdx.x;
  const long long off = token_offset(pg, seq, first + j);
  if (off < 0 && threadIdx.x == 0 && status) atomicCAS(status, 0, (ST_BAD_ARG << 24) | 0x6a7);
  for (int c = threadIdx.x * 8; c < pg.width; c += blockDim.x * 8) {
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (off >= 0) load8((const T*)pg.pool + off + c, v);
    store8(out + j * ldo + c, v);
  }
}

// one thread per (row, V pairs, G heads): the angles are worked out once for its heads
template <typename T, int V, int G>
__global__ void __launch_bounds__(128)
rotate_heads_kernel(T* __restrict__ q, long long ldq, int rows, int heads, int head_pitch, int off, int half,
                    const float* __restrict__ freq, RowPos rp) {
  const int chunks = half / V, groups = (heads + G - 1) / G;
  const long long t = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int i = (int)(t % chunks) * V, h0 = (int)(t / chunks % groups) * G, row = (int)(t / ((long long)chunks * groups));
  if (row >= rows) return;
  int seq;
  const int pos = row_position(rp, row, seq);
  T* p = q + row * ldq + (long long)h0 * head_pitch + off + i;
  float a[G][V], b[G][V];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    if (h0 + g >= heads) continue;
    if constexpr (V == 8) {
      load8(p + g * head_pitch, a[g]);
      load8(p + g * head_pitch + half, b[g]);
    } else {
      a[g][0] = to_f(p[g * head_pitch]); b[g][0] = to_f(p[g * head_pitch + half]);
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) {
    float sn, cs;
    sincosf((float)pos * freq[i + j], &sn, &cs);
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const float u = a[g][j], v = b[g][j];
      a[g][j] = u * cs - v * sn;
      b[g][j] = v * cs + u * sn;
    }
  }
#pragma unroll
  for (int g = 0; g < G; ++g) {
    if (h0 + g >= heads) continue;
    if constexpr (V == 8) {
      store8(p + g * head_pitch, a[g]);
      store8(p + g * head_pitch + half, b[g]);
    } else {
      p[g * head_pitch] = from_f<T>(a[g][0]); p[g * head_pitch + half] = from_f<T>(b[g][0]);
    }
  }
}

// ----------------------------------------------------------------------------- absorb
// grid (ceil(kvp / 128), heads, rows), 256 threads: 16 threads cover 128 latent entries, 16 groups split the head dim
template <typename T>
__global__ void __launch_bounds__(256)
absorb_query_kernel(const T* __restrict__ q, long long ldq, int heads, int head_pitch, int dp, const T* __restrict__ Wuk,
                    int kvp, T* __restrict__ qa) {
  __shared__ float part[16][128 + 4];
  const int h = blockIdx.y, row = blockIdx.z;
  const int kk = (threadIdx.x & 15) * 8, g = threadIdx.x >> 4;
  const int k = blockIdx.x * 128 + kk;
  const T* w = Wuk + (long long)h * dp * kvp + k;
  Raw8<T> first;
  const bool any = k < kvp && g < dp;
  if (any) first = raw8(w + (long long)g * kvp);
  pdl_wait();
  pdl_trigger();
  const T* qh = q + row * ldq + (long long)h * head_pitch;
  float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  if (any) {
    float f[8];
    unraw8(first, f);
    float qd = to_f(qh[g]);
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] += qd * f[j];
#pragma unroll 4
    for (int d = g + 16; d < dp; d += 16) {
      unraw8(raw8(w + (long long)d * kvp), f);
      qd = to_f(qh[d]);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] += qd * f[j];
    }
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) part[g][kk + j] = acc[j];
  __syncthreads();
  if (threadIdx.x < 128 && (int)(blockIdx.x * 128 + threadIdx.x) < kvp) {
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < 16; ++i) v += part[i][threadIdx.x];
    qa[((long long)row * heads + h) * kvp + blockIdx.x * 128 + threadIdx.x] = from_f<T>(v);
  }
}

// -------------------------------------------------------------------------- attention
// Plain form. grid (splits, heads, rows), 128 threads; dynamic shared memory: W + kvp floats.
template <typename T>
__global__ void __launch_bounds__(128)
latent_attention_kernel(const LatentAttn d) {
  extern __shared__ float sm[];
  __shared__ float s_p[128];
  __shared__ long long s_off[128];
  __shared__ float s_red[8];
  const int split = blockIdx.x, h = blockIdx.y, row = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int W = d.kvp + d.rp;
  float* sq = sm;                 // [W] absorbed query | rotated part
  float* so = sm + W;             // [kvp]
  pdl_wait();
  pdl_trigger();
  int seq;
  const int pos = row_position(d.pos, row, seq);
  const KeyRange kr = split_keys(pos, d.window, d.splits, split, 1);
  const long long slot = ((long long)row * d.heads + h) * d.splits + split;
  if (kr.begin >= kr.end) {
    if (tid == 0) { d.ml[slot * 2] = NEG_BIG; d.ml[slot * 2 + 1] = 0.f; }
    return;
  }
  const T* qa = (const T*)d.qa + ((long long)row * d.heads + h) * d.kvp;
  const T* qr = (const T*)d.q + row * d.ldq + (long long)h * d.head_pitch + d.dp;
  for (int c = tid; c < d.kvp; c += 128) { sq[c] = to_f(qa[c]); so[c] = 0.f; }
  const int half = d.dims >> 1;
  for (int i = tid; i < d.rp; i += 128) {
    float v = i < d.rot_dim ? to_f(qr[i]) : 0.f;
    if (i < d.dims) {
      const int p = i < half ? i : i - half;
      float sn, cs;
      sincosf((float)pos * d.freq[p], &sn, &cs);
      const float a = to_f(qr[p]), b = to_f(qr[p + half]);
      v = i < half ? a * cs - b * sn : b * cs + a * sn;
    }
    sq[d.kvp + i] = v;
  }
  const float sc = d.scale * 1.4426950408889634f;
  float M = NEG_BIG, L = 0.f;
  for (int tile = kr.begin; tile < kr.end; tile += 128) {
    __syncthreads();
    const int j = tile + tid;
    float s = NEG_BIG;
    long long off = -1;
    if (j < kr.end) {
      off = token_offset(d.pg, seq, j);
      if (off >= 0) {
        const T* e = (const T*)d.pg.pool + off;
        float a = 0.f;
        for (int c = 0; c < W; c += 8) {
          float f[8];
          load8(e + c, f);
#pragma unroll
          for (int i = 0; i < 8; ++i) a += f[i] * sq[c + i];
        }
        s = a * sc;
      }
    }
    s_off[tid] = off;
    float mx = warp_max(s);
    if (lane == 0) s_red[warp] = mx;
    __syncthreads();
    const float m_new = fmaxf(M, fmaxf(fmaxf(s_red[0], s_red[1]), fmaxf(s_red[2], s_red[3])));
    const float p = off >= 0 ? exp2f(s - m_new) : 0.f;
    s_p[tid] = p;
    const float ps = warp_sum(p);
    if (lane == 0) s_red[4 + warp] = ps;
    __syncthreads();
    const float alpha = exp2f(M - m_new);
    L = L * alpha + (s_red[4] + s_red[5]) + (s_red[6] + s_red[7]);
    const int cnt = min(128, kr.end - tile);
    for (int c = tid; c < d.kvp; c += 128) {
      float o = so[c] * alpha;
      for (int k = 0; k < cnt; ++k)
        if (s_off[k] >= 0) o += s_p[k] * to_f(((const T*)d.pg.pool)[s_off[k] + c]);
      so[c] = o;
    }
    M = m_new;
  }
  if (tid == 0) { d.ml[slot * 2] = M; d.ml[slot * 2 + 1] = L; }
  for (int c = tid; c < d.kvp; c += 128) d.acc[slot * d.kvp + c] = so[c];
}

// Tensor-core form: grid (splits, ceil(heads / 16), rows), 256 threads. Each of the eight warps scores eight of a tile's
// keys, then owns every eighth 16-column unit of the weighted latents.
constexpr int KT = 64;                       // keys per tile
constexpr int AW = 8;                        // warps
__host__ __device__ constexpr int padded_width(int W) { return (W + 31) / 32 * 32; }      // scores step through 32 columns
inline size_t mma_smem_bytes(int W) { return (size_t)(16 + KT) * (padded_width(W) + 8) * 2 + (size_t)16 * (KT + 8) * 2; }

// NU: 16-column units of the latent per warp (kvp <= 128 * NU)
template <int NU>
__global__ void __launch_bounds__(AW * 32)
latent_attention_mma_kernel(const LatentAttn d) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float s_max[AW][16];
  __shared__ float s_sum[AW][16];
  const int split = blockIdx.x, h0 = blockIdx.y * 16, row = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int W = d.kvp + d.rp, WP = padded_width(W), LD = WP + 8, LP = KT + 8;
  bf16* sQ = reinterpret_cast<bf16*>(smem_raw);
  bf16* sK = sQ + 16 * LD;
  bf16* sP = sK + KT * LD;
  const int half = d.dims >> 1;
  if (WP > W) {                                                 // columns that only fill up the last step
    for (int i = tid; i < (16 + KT) * 2; i += AW * 32)
      *reinterpret_cast<uint4*>(sQ + (i >> 1) * LD + W + (i & 1) * 8) = make_uint4(0, 0, 0, 0);
  }
  pdl_wait();
  pdl_trigger();
  int seq;
  const int pos = row_position(d.pos, row, seq);
  const KeyRange kr = split_keys(pos, d.window, d.splits, split, KT);
  if (kr.begin >= kr.end) {
    if (tid < 16 && h0 + tid < d.heads) {
      const long long slot = ((long long)row * d.heads + h0 + tid) * d.splits + split;
      d.ml[slot * 2] = NEG_BIG; d.ml[slot * 2 + 1] = 0.f;
    }
    return;
  }
  auto load_tile = [&](int tile) {
    const int mine = tile + warp * 8 + (lane & 7);              // the warp's eight keys: addresses first, then the copies
    const long long my_off = mine < kr.end ? token_offset(d.pg, seq, mine) : -1;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const long long off = __shfl_sync(0xffffffffu, my_off, k);
      bf16* dst = sK + (warp * 8 + k) * LD;
      if (off >= 0) {
        const bf16* src = (const bf16*)d.pg.pool + off;
        for (int c = lane * 8; c < W; c += 256) cp_async16(dst + c, src + c);
      } else {
        for (int c = lane * 8; c < W; c += 256) *reinterpret_cast<uint4*>(dst + c) = make_uint4(0, 0, 0, 0);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_tile(kr.begin);
  for (int h = warp; h < 16; h += AW) {
    const bool on = h0 + h < d.heads;
    const bf16* qa = (const bf16*)d.qa + ((long long)row * d.heads + h0 + h) * d.kvp;
    for (int c = lane * 8; c < d.kvp; c += 256)
      *reinterpret_cast<uint4*>(sQ + h * LD + c) = on ? *reinterpret_cast<const uint4*>(qa + c) : make_uint4(0, 0, 0, 0);
    const bf16* qr = (const bf16*)d.q + row * d.ldq + (long long)(h0 + h) * d.head_pitch + d.dp;
    bf16* dst = sQ + h * LD + d.kvp;
    for (int i = lane; i < half; i += 32) {
      float sn, cs;
      sincosf((float)pos * d.freq[i], &sn, &cs);
      const float a = on ? to_f(qr[i]) : 0.f, b = on ? to_f(qr[i + half]) : 0.f;
      dst[i] = __float2bfloat16_rn(a * cs - b * sn);
      dst[i + half] = __float2bfloat16_rn(b * cs + a * sn);
    }
    for (int i = d.dims + lane; i < d.rp; i += 32) dst[i] = on && i < d.rot_dim ? qr[i] : __float2bfloat16_rn(0.f);
  }
  const float sc = d.scale * 1.4426950408889634f;
  float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.f, 0.f};
  float o[NU][2][4];
#pragma unroll
  for (int u = 0; u < NU; ++u)
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[u][t][e] = 0.f;
  const int units = d.kvp / 16;
  for (int tile = kr.begin; tile < kr.end; tile += KT) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // scores of 16 heads x this warp's 8 keys, even and odd steps in accumulators of their own
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const bf16* qp = sQ + (lane & 15) * LD + (lane >> 4) * 8;
    const bf16* kp = sK + (warp * 8 + (lane & 7)) * LD + (lane >> 3) * 8;
#pragma unroll 4
    for (int k = 0; k < WP; k += 32) {
      uint32_t a0[4], a1[4], b[4];
      ldmatrix4(a0, qp + k);
      ldmatrix4(a1, qp + k + 16);
      ldmatrix4(b, kp + k);
      mma_16816(s[0], a0, b[0], b[1]);
      mma_16816(s[1], a1, b[2], b[3]);
    }
    const int j = tile + warp * 8 + (lane & 3) * 2;             // this lane's keys: j, j + 1
    float mx[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
#pragma unroll
      for (int e = 0; e < 2; ++e) s[0][r * 2 + e] = j + e < kr.end ? (s[0][r * 2 + e] + s[1][r * 2 + e]) * sc : NEG_BIG;
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
    // weighted latents: this warp's column units
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
          ldmatrix4_trans(b, sK + (k + (lane & 15)) * LD + unit * 16 + (lane >> 4) * 8);
          mma_16816(o[u][0], a, b[0], b[1]);
          mma_16816(o[u][1], a, b[2], b[3]);
        }
      }
    }
    if (tile + KT < kr.end) {
      __syncthreads();                                          // the tile's keys and weights have been read
      load_tile(tile + KT);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    if ((lane & 3) == 0) s_sum[warp][(lane >> 2) + r * 8] = l_run[r];
    const int h = h0 + (lane >> 2) + r * 8;
    if (h >= d.heads) continue;
    const long long slot = ((long long)row * d.heads + h) * d.splits + split;
    if (warp == 0 && (lane & 3) == 0) d.ml[slot * 2] = m_run[r];
    float* dst = d.acc + slot * d.kvp;
#pragma unroll
    for (int u = 0; u < NU; ++u) {
      const int unit = warp + u * AW;
      if (unit >= units) continue;
#pragma unroll
      for (int t = 0; t < 2; ++t)
        *reinterpret_cast<float2*>(dst + unit * 16 + t * 8 + (lane & 3) * 2) = make_float2(o[u][t][r * 2], o[u][t][r * 2 + 1]);
    }
  }
  __syncthreads();
  if (tid < 16 && h0 + tid < d.heads) {
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < AW; ++w) l += s_sum[w][tid];
    d.ml[(((long long)row * d.heads + h0 + tid) * d.splits + split) * 2 + 1] = l;
  }
}

// grid (ceil(vp / 16), heads, rows), 256 threads, two outputs per warp; dynamic shared memory: kvp floats
template <typename T>
__global__ void __launch_bounds__(256)
latent_values_kernel(const float* __restrict__ ml, const float* __restrict__ acc, int heads, int splits, int kvp,
                     const T* __restrict__ Wuv, int vp, T* __restrict__ y, long long ldy, NextWeights next) {
  constexpr int OUT = 2, AHEAD = 2;                 // outputs per warp, 256-column chunks requested before the wait
  extern __shared__ float lat[];
  __shared__ float s_w[MAX_SPLITS];
  const int h = blockIdx.y, row = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int j0 = blockIdx.x * (8 * OUT) + warp * OUT;
  prefetch_l2_slice(next, blockIdx.x + (long long)gridDim.x * blockIdx.y, (long long)gridDim.x * gridDim.y);
  const T* w = Wuv + ((long long)h * vp + j0) * kvp + lane * 8;
  Raw8<T> first[AHEAD][OUT];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i)
#pragma unroll
    for (int r = 0; r < OUT; ++r)
      if (j0 + r < vp && i * 256 + lane * 8 < kvp) first[i][r] = raw8(w + (long long)r * kvp + i * 256);
  pdl_wait();
  pdl_trigger();
  const long long slot = ((long long)row * heads + h) * splits;
  if (warp == 0) {                                  // a lane per split: its weight in the combination
    const float m = lane < splits ? ml[(slot + lane) * 2] : NEG_BIG, l = lane < splits ? ml[(slot + lane) * 2 + 1] : 0.f;
    const float M = warp_max(l > 0.f ? m : NEG_BIG);
    const float f = l > 0.f ? exp2f(m - M) : 0.f;
    const float L = warp_sum(l * f);
    s_w[lane] = L > 0.f ? f / L : 0.f;
  }
  __syncthreads();
  for (int c = threadIdx.x; c < kvp; c += 256) {
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < splits; ++s) {
      const float f = s_w[s];                       // an empty split leaves its sums unwritten
      const float t = f > 0.f ? acc[(slot + s) * kvp + c] : 0.f;
      v += f * t;
    }
    lat[c] = v;
  }
  __syncthreads();
  float sum[OUT] = {0.f, 0.f};
  auto dot = [&](const Raw8<T>& raw, int r, int c) {
    float f[8];
    unraw8(raw, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) sum[r] += f[i] * lat[c + lane * 8 + i];
  };
#pragma unroll
  for (int i = 0; i < AHEAD; ++i)
#pragma unroll
    for (int r = 0; r < OUT; ++r)
      if (j0 + r < vp && i * 256 + lane * 8 < kvp) dot(first[i][r], r, i * 256);
  for (int c = AHEAD * 256; c + lane * 8 < kvp; c += 256) {
#pragma unroll
    for (int r = 0; r < OUT; ++r)
      if (j0 + r < vp) dot(raw8(w + (long long)r * kvp + c), r, c);
  }
#pragma unroll
  for (int r = 0; r < OUT; ++r) {
    const float v = warp_sum(sum[r]);
    if (lane == 0 && j0 + r < vp) y[row * ldy + (long long)h * vp + j0 + r] = from_f<T>(v);
  }
}

bool pages_ok(const Pages& p) {
  return p.pool && p.table && p.max_pages > 0 && p.shift >= 0 && p.shift <= 16 && p.n_pages > 0 && p.width > 0 && !(p.width & 7);
}
bool rows_ok(const RowPos& p) { return p.lens && p.per_seq > 0; }

}  // namespace

cudaError_t latent_post(const LatentPost& d, int* status, cudaStream_t s) {
  if (d.rows <= 0 || !pages_ok(d.pg) || !rows_ok(d.pos) || d.pg.width != d.kvp + d.rp || d.kv_rank > d.kvp || d.kv_rank <= 0 ||
      d.dims > d.rot_dim || d.rot_dim > d.rp || (d.dims & 1) || d.q_rank > d.qp || (d.f32 && !d.z_f32))
    return cudaErrorInvalidValue;
  const dim3 grid(d.rows, d.cq ? 2 : 1);
  if (d.f32) latent_post_kernel<float, float><<<grid, 128, 0, s>>>(d, status);
  else if (d.z_f32) latent_post_kernel<bf16, float><<<grid, 128, 0, s>>>(d, status);
  else latent_post_kernel<bf16, bf16><<<grid, 128, 0, s>>>(d, status);
  return cudaGetLastError();
}

cudaError_t latent_gather(bool f32, const Pages& pg, int seq, int first, int count, void* out, long long ldo,
                          int* status, cudaStream_t s) {
  if (count <= 0 || first < 0 || seq < 0 || !pages_ok(pg) || (ldo & 7) || ldo < pg.width) return cudaErrorInvalidValue;
  if (f32) latent_gather_kernel<float><<<count, 128, 0, s>>>(pg, seq, first, (float*)out, ldo, status);
  else latent_gather_kernel<bf16><<<count, 128, 0, s>>>(pg, seq, first, (bf16*)out, ldo, status);
  return cudaGetLastError();
}

cudaError_t rotate_heads(bool f32, void* q, long long ldq, int rows, int heads, int head_pitch, int off, int dims,
                         const float* freq, const RowPos& pos, cudaStream_t s) {
  if (rows <= 0 || heads <= 0 || dims < 0 || (dims & 1) || off + dims > head_pitch || (long long)heads * head_pitch > ldq || !rows_ok(pos))
    return cudaErrorInvalidValue;
  if (dims == 0) return cudaSuccess;
  const int half = dims / 2;
  const bool vec = half % 8 == 0 && off % 8 == 0 && head_pitch % 8 == 0 && ldq % 8 == 0;
  constexpr int G = 4;
  const long long n = (long long)rows * ((heads + G - 1) / G) * (half / (vec ? 8 : 1));
  const dim3 grid((unsigned)((n + 127) / 128));
  if (f32) {
    auto k = vec ? rotate_heads_kernel<float, 8, G> : rotate_heads_kernel<float, 1, G>;
    k<<<grid, 128, 0, s>>>((float*)q, ldq, rows, heads, head_pitch, off, half, freq, pos);
  } else {
    auto k = vec ? rotate_heads_kernel<bf16, 8, G> : rotate_heads_kernel<bf16, 1, G>;
    k<<<grid, 128, 0, s>>>((bf16*)q, ldq, rows, heads, head_pitch, off, half, freq, pos);
  }
  return cudaGetLastError();
}

cudaError_t absorb_query(bool f32, const void* q, long long ldq, int rows, int heads, int head_pitch, int dp,
                         const void* Wuk, int kvp, void* qa, bool pdl, cudaStream_t s) {
  if (rows <= 0 || rows > 65535 || heads <= 0 || heads > 65535 || dp <= 0 || dp > head_pitch || kvp <= 0 || (kvp & 7))
    return cudaErrorInvalidValue;
  const dim3 grid((kvp + 127) / 128, heads, rows);
  if (f32) return launch(pdl, absorb_query_kernel<float>, grid, dim3(256), 0, s, (const float*)q, ldq, heads, head_pitch, dp, (const float*)Wuk, kvp, (float*)qa);
  return launch(pdl, absorb_query_kernel<bf16>, grid, dim3(256), 0, s, (const bf16*)q, ldq, heads, head_pitch, dp, (const bf16*)Wuk, kvp, (bf16*)qa);
}

bool latent_attention_tensor_cores(const LatentAttn& d) {
  return !d.f32 && !(d.kvp & 15) && !(d.rp & 15) && d.kvp <= 512 && mma_smem_bytes(d.kvp + d.rp) <= 200 * 1024;
}

template <int NU>
static cudaError_t launch_mma(const LatentAttn& d, cudaStream_t s) {
  static PerDeviceOnce configured;
  const cudaError_t ce = configured.once([] {
    return cudaFuncSetAttribute(latent_attention_mma_kernel<NU>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  });
  if (ce != cudaSuccess) return ce;
  return launch(d.pdl, latent_attention_mma_kernel<NU>, dim3(d.splits, (d.heads + 15) / 16, d.rows), dim3(AW * 32),
                mma_smem_bytes(d.kvp + d.rp), s, d);
}

cudaError_t latent_attention(const LatentAttn& d, cudaStream_t s) {
  if (d.rows <= 0 || d.rows > 65535 || d.heads <= 0 || d.heads > 65535 || d.splits <= 0 || d.splits > MAX_SPLITS || !pages_ok(d.pg) || !rows_ok(d.pos) ||
      d.pg.width != d.kvp + d.rp || (d.kvp & 7) || (d.rp & 7) || d.dims > d.rot_dim || d.rot_dim > d.rp || (d.dims & 1) ||
      d.dp + d.rot_dim > d.head_pitch)
    return cudaErrorInvalidValue;
  if (latent_attention_tensor_cores(d)) {
    if (d.kvp <= 128) return launch_mma<1>(d, s);
    if (d.kvp <= 256) return launch_mma<2>(d, s);
    return launch_mma<4>(d, s);
  }
  const size_t smem = (size_t)(2 * d.kvp + d.rp) * sizeof(float);
  if (smem > 40 * 1024) return cudaErrorInvalidValue;
  const dim3 grid(d.splits, d.heads, d.rows);
  if (d.f32) return launch(d.pdl, latent_attention_kernel<float>, grid, dim3(128), smem, s, d);
  return launch(d.pdl, latent_attention_kernel<bf16>, grid, dim3(128), smem, s, d);
}

cudaError_t latent_values(bool f32, const float* ml, const float* acc, int rows, int heads, int splits, int kvp,
                          const void* Wuv, int vp, void* y, long long ldy, bool pdl, const NextWeights& next,
                          cudaStream_t s) {
  if (rows <= 0 || rows > 65535 || heads <= 0 || heads > 65535 || splits <= 0 || splits > MAX_SPLITS || kvp <= 0 || (kvp & 7) || vp <= 0 || kvp > 10240)
    return cudaErrorInvalidValue;
  const dim3 grid((vp + 15) / 16, heads, rows);
  const size_t smem = (size_t)kvp * sizeof(float);
  if (f32) return launch(pdl, latent_values_kernel<float>, grid, dim3(256), smem, s, ml, acc, heads, splits, kvp, (const float*)Wuv, vp, (float*)y, ldy, next);
  return launch(pdl, latent_values_kernel<bf16>, grid, dim3(256), smem, s, ml, acc, heads, splits, kvp, (const bf16*)Wuv, vp, (bf16*)y, ldy, next);
}

}  // namespace serve
}  // namespace nc
