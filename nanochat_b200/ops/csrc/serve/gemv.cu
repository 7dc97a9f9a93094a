// Matrix-vector products of a decode step (up to 8 rows, bf16 weights) on mma.sync.
//
// The 16 x 8 x 16 tile fits the problem: 16 outputs x 8 rows of the step. A weight fragment is loaded straight from
// global memory with 16-byte loads: the sum over k does not care about order, so lane group q of a warp takes the eight
// neighbouring elements k0 + 8q .. k0 + 8q + 7 of its output's weight row and feeds them to two MMAs, the activations being
// picked by the same rule. Eight warps split K; their tiles are summed through shared memory. The tensor cores make the
// arithmetic disappear, so the time of a product is the time of its bytes whatever the number of rows.
//
//   gemv            one product; input norm (linear once the row statistic is known: the statistic rides along), gated
//                   residual update of the output, extra CTAs that append the step's entries to the latent store
//                   Few outputs and a long K: four CTAs of a cluster share K and add up over distributed shared memory
//   gemv_relu_glu   gate and up product of a dense feed-forward with its activation
//   expert_*_rows   a step's experts: every chosen expert's weights are read once for all rows that chose it (down: the
//                   four CTAs of a cluster take every fourth expert)
#include <cooperative_groups.h>

#include "latent_store.cuh"

namespace nc {
namespace serve {

namespace {

constexpr int WARPS = 8;
constexpr int THREADS = WARPS * 32;
constexpr int ROWS = 8;               // rows of a step one MMA takes

__device__ __forceinline__ void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// Weight fragments of MT 16-output tiles for U k-steps of 32: rows n and n + 8 of each tile, eight elements each.
template <int MT, int U>
struct Frag {
  uint4 lo[U][MT], hi[U][MT];
};

// A block's tiles: row pointers of this lane (already offset by its k group), null past the last output.
template <int MT>
struct TileRows {
  const bf16* lo[MT];
  const bf16* hi[MT];
};

template <int MT, int U>
__device__ __forceinline__ void load_frag(Frag<MT, U>& f, const TileRows<MT>& w, int k0, int q8, int K) {
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int k = k0 + u * (WARPS * 32);
    const bool in = k + q8 < K;
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      f.lo[u][t] = in && w.lo[t] ? ld_once(w.lo[t] + k) : make_uint4(0, 0, 0, 0);
      f.hi[u][t] = in && w.hi[t] ? ld_once(w.hi[t] + k) : make_uint4(0, 0, 0, 0);
    }
  }
}

template <int MT, int U, class X>
__device__ __forceinline__ void mma_frag(float (&acc)[MT][4], const Frag<MT, U>& f, int k0, int q8, int K, X& x) {
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int k = k0 + u * (WARPS * 32) + q8;
    const uint4 b = k < K ? x(k) : make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      mma_16816(acc[t], f.lo[u][t].x, f.hi[u][t].x, f.lo[u][t].y, f.hi[u][t].y, b.x, b.y);
      mma_16816(acc[t], f.lo[u][t].z, f.hi[u][t].z, f.lo[u][t].w, f.hi[u][t].w, b.z, b.w);
    }
  }
}

template <int MT>
__device__ __forceinline__ TileRows<MT> tile_rows(const bf16* W, long long ldw, int n0, int N, int lane) {
  TileRows<MT> r;
  const int n = n0 + (lane >> 2), q8 = (lane & 3) * 8;
#pragma unroll
  for (int t = 0; t < MT; ++t) {
    r.lo[t] = n + t * 16 < N ? W + (long long)(n + t * 16) * ldw + q8 : nullptr;
    r.hi[t] = n + t * 16 + 8 < N ? W + (long long)(n + t * 16 + 8) * ldw + q8 : nullptr;
  }
  return r;
}

// Tiles of the eight warps to shared memory: s[warp][output][row].
template <int MT>
__device__ __forceinline__ void spill_tiles(const float (&acc)[MT][4], float (*s)[MT * 16][ROWS + 1], int warp, int lane) {
#pragma unroll
  for (int t = 0; t < MT; ++t) {
    const int m = t * 16 + (lane >> 2), n = (lane & 3) * 2;
    s[warp][m][n] = acc[t][0]; s[warp][m][n + 1] = acc[t][1];
    s[warp][m + 8][n] = acc[t][2]; s[warp][m + 8][n + 1] = acc[t][3];
  }
}

constexpr int CLUSTER = 4;

// The CTA's tile (outputs x rows), summed over its warps, then over the cluster; the result is valid in the cluster's first
// CTA. All threads of all CTAs of the cluster call this.
template <int M>
__device__ __forceinline__ float cluster_total(float (*s_acc)[M][ROWS + 1], float (*s_part)[ROWS], bool mine, int m, int b) {
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  float v = 0.f;
  if (mine) {
#pragma unroll
    for (int i = 0; i < WARPS; ++i) v += s_acc[i][m][b];
    s_part[m][b] = v;
  }
  cluster.sync();
  if (mine && cluster.block_rank() == 0) {
#pragma unroll
    for (int r = 1; r < CLUSTER; ++r) v += cluster.map_shared_rank(&s_part[0][0], r)[m * ROWS + b];
  }
  cluster.sync();                       // the others' shared memory stays until it has been read
  return v;
}

struct GemvArgs {
  const void* x; long long ldx;
  const float* w; float eps; int n_real;
  const bf16* W; long long ldw;
  int B, N, K, epi, accumulate;
  void* out; long long ldo;
  float* resid; long long ldr; const float* g; long long ldg; const float* bias; float mult; const float* extra;
  bf16* h_out; long long ldh;
  NextWeights next;
  LatentStore store;
  int n_blocks;
};

// SPLIT: CTAs of a cluster (grid y) that share K; 1 or CLUSTER
template <bool NORM, int MT, int SPLIT>
__device__ __forceinline__ void gemv_body(const GemvArgs& a) {
  static_assert(SPLIT == 1 || (!NORM && SPLIT == CLUSTER), "only plain products share K");
  constexpr int U = MT == 1 ? 4 : 2;
  constexpr int STEP = U * WARPS * 32;
  __shared__ float s_part[SPLIT > 1 ? MT * 16 : 1][ROWS];
  __shared__ float s_acc[WARPS][MT * 16][ROWS + 1];
  __shared__ float s_ss[WARPS][ROWS];
  __shared__ float s_red[32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (NORM && (int)blockIdx.x >= a.n_blocks) {              // extra CTAs: append to the latent store
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
  const int n0 = blockIdx.x * (MT * 16), q8 = (lane & 3) * 8, row = lane >> 2;
  // grid y without a split: groups of eight rows (plain stores only)
  const int group = SPLIT == 1 ? (int)blockIdx.y : 0, B = SPLIT == 1 ? min(ROWS, a.B - group * ROWS) : a.B;
  if (blockIdx.y == 0) prefetch_l2_slice(a.next, blockIdx.x, a.n_blocks);
  const TileRows<MT> w = tile_rows<MT>(a.W, a.ldw, n0, a.N, lane);
  Frag<MT, U> f;
  const int k_first = warp * 32 + (SPLIT > 1 ? (int)blockIdx.y * STEP : 0);
  load_frag(f, w, k_first, q8, a.K);               // weights do not depend on the kernel before
  pdl_wait();
  pdl_trigger();
  float acc[MT][4], ss = 0.f;
#pragma unroll
  for (int t = 0; t < MT; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[t][e] = 0.f;
  const float* xf = (const float*)a.x + row * a.ldx;
  const bf16* xb = (const bf16*)a.x + (group * ROWS + row) * a.ldx;
  auto x = [&](int k) -> uint4 {
    if (row >= B) return make_uint4(0, 0, 0, 0);
    if (!NORM) return *reinterpret_cast<const uint4*>(xb + k);
    float v[8], nw[8];
    load8(xf + k, v);
    load8(a.w + k, nw);
#pragma unroll
    for (int j = 0; j < 8; ++j) { ss += v[j] * v[j]; v[j] *= nw[j]; }
    return make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  };
  for (int k0 = k_first; k0 < a.K;) {
    mma_frag(acc, f, k0, q8, a.K, x);
    k0 += SPLIT * STEP;
    if (k0 < a.K) load_frag(f, w, k0, q8, a.K);
  }
  spill_tiles<MT>(acc, s_acc, warp, lane);
  if (NORM) {
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    if ((lane & 3) == 0) s_ss[warp][row] = ss;
  }
  __syncthreads();
  auto scale = [&](int b) {
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < WARPS; ++i) t += s_ss[i][b];
    return inv_rms(t, a.n_real, a.eps);
  };
  if (NORM && a.h_out != nullptr && blockIdx.x == 0) {
    for (int b = 0; b < a.B; ++b) {
      const float r = scale(b);
      for (int k = tid * 8; k < a.K; k += THREADS * 8) {
        float v[8], nw[8];
        load8((const float*)a.x + b * a.ldx + k, v);
        load8(a.w + k, nw);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= r * nw[j];
        store8(a.h_out + b * a.ldh + k, v);
      }
    }
  }
  const int m = tid & (MT * 16 - 1), b = tid / (MT * 16), n = n0 + m;
  float v = 0.f;
  if constexpr (SPLIT > 1) {
    v = cluster_total<MT * 16>(s_acc, s_part, tid < MT * 16 * ROWS, m, b);
    if (blockIdx.y != 0) return;
  }
  if (tid < MT * 16 * ROWS) {
    if (b < B && n < a.N) {
      if constexpr (SPLIT == 1) {
#pragma unroll
        for (int i = 0; i < WARPS; ++i) v += s_acc[i][m][b];
      }
      if (NORM) v *= scale(b);
      if (a.epi == GEMV_STORE_F32) {
        ((float*)a.out)[(group * ROWS + b) * a.ldo + n] = v;
      } else if (a.epi == GEMV_STORE_BF16) {
        ((bf16*)a.out)[(group * ROWS + b) * a.ldo + n] = __float2bfloat16_rn(v);
      } else {
        float r = a.mult * sigmoidf(a.g[b * a.ldg + n] + a.bias[n]) * v;
        if (a.extra) r += a.extra[b * a.ldr + n];
        if (a.accumulate) r += a.resid[b * a.ldr + n];
        a.resid[b * a.ldr + n] = r;
      }
    }
  }
}

template <bool NORM, int MT>
__global__ void __launch_bounds__(THREADS) gemv_kernel(const GemvArgs a) { gemv_body<NORM, MT, 1>(a); }
__global__ void __cluster_dims__(1, CLUSTER, 1) __launch_bounds__(THREADS) gemv_cluster_kernel(const GemvArgs a) {
  gemv_body<false, 1, CLUSTER>(a);
}

// Gate and up rows of the same outputs as the two tiles of a CTA; the activation closes the product.
__global__ void __launch_bounds__(THREADS) gemv_relu_glu_kernel(const GemvArgs a) {
  constexpr int U = 2;
  __shared__ float s_acc[WARPS][32][ROWS + 1];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n0 = blockIdx.x * 16, q8 = (lane & 3) * 8, row = lane >> 2;
  prefetch_l2_slice(a.next, blockIdx.x, a.n_blocks);
  const TileRows<1> wg = tile_rows<1>(a.W, a.ldw, n0, a.N, lane), wu = tile_rows<1>(a.W + a.N * a.ldw, a.ldw, n0, a.N, lane);
  const TileRows<2> w = {{wg.lo[0], wu.lo[0]}, {wg.hi[0], wu.hi[0]}};
  Frag<2, U> f;
  load_frag(f, w, warp * 32, q8, a.K);
  pdl_wait();
  pdl_trigger();
  float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
  const bf16* xb = (const bf16*)a.x + row * a.ldx;
  auto x = [&](int k) -> uint4 { return row < a.B ? *reinterpret_cast<const uint4*>(xb + k) : make_uint4(0, 0, 0, 0); };
  for (int k0 = warp * 32; k0 < a.K;) {
    mma_frag(acc, f, k0, q8, a.K, x);
    k0 += U * WARPS * 32;
    if (k0 < a.K) load_frag(f, w, k0, q8, a.K);
  }
  spill_tiles<2>(acc, s_acc, warp, lane);
  __syncthreads();
  if (tid < 16 * ROWS) {
    const int m = tid & 15, b = tid >> 4, n = n0 + m;
    if (b < a.B && n < a.N) {
      float g = 0.f, u = 0.f;
#pragma unroll
      for (int i = 0; i < WARPS; ++i) { g += s_acc[i][m][b]; u += s_acc[i][m + 16][b]; }
      ((bf16*)a.out)[b * a.ldo + n] = __float2bfloat16_rn(fmaxf(g, 0.f) * u);
    }
  }
}

// ----------------------------------------------------------------------------- experts
// The step's choices (rows * top of them) in shared memory, with the position of each expert's first mention and how
// many distinct experts were mentioned before it.
constexpr int MAX_CHOICES = 512;
struct Choices {
  int idx[MAX_CHOICES];
  short first[MAX_CHOICES];            // first mention of the same expert
  short order[MAX_CHOICES];            // distinct experts before it (first mentions only)
  int distinct;
};
__device__ __forceinline__ void load_choices(Choices& c, const int* idx, int n) {
  for (int i = threadIdx.x; i < n; i += blockDim.x) c.idx[i] = idx[i];
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    int j = 0;
    while (c.idx[j] != c.idx[i]) ++j;
    c.first[i] = (short)j;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    int k = 0;
    for (int j = 0; j < i; ++j) k += c.first[j] == j;
    c.order[i] = (short)k;
    if (i == n - 1) c.distinct = k + (c.first[i] == i);
  }
  __syncthreads();
}

struct ExpertArgs {
  const bf16* in; long long ldin;      // gate_up: the rows' h; down: act (choices x fp)
  int B, top, K, N;                    // N: outputs (fp for gate_up)
  const bf16* W;                       // experts x (2 fp | N) x K
  const int* idx; const float* wt;
  bf16* act;
  float* out; long long ldo; const float* g; long long ldg; const float* bias; float mult; const float* extra;
};

// grid (distinct experts at most, ceil(fp / 16)): act of every row that chose this CTA's expert
__global__ void __launch_bounds__(THREADS)
expert_gate_up_rows_kernel(const ExpertArgs a) {
  constexpr int U = 2;
  __shared__ Choices c;
  __shared__ float s_acc[WARPS][32][ROWS + 1];
  __shared__ int s_choice[ROWS], s_first;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = a.B * a.top;
  if (tid < ROWS) s_choice[tid] = -1;
  pdl_wait();
  pdl_trigger();
  load_choices(c, a.idx, n);
  if ((int)blockIdx.x >= c.distinct) return;
  for (int i = tid; i < n; i += THREADS)
    if (c.order[c.first[i]] == (int)blockIdx.x) { s_choice[i / a.top] = i; s_first = c.first[i]; }
  __syncthreads();
  const int n0 = blockIdx.y * 16, q8 = (lane & 3) * 8, choice = s_choice[lane >> 2];
  const bf16* We = a.W + (long long)c.idx[s_first] * 2 * a.N * a.K;
  const TileRows<1> wg = tile_rows<1>(We, a.K, n0, a.N, lane), wu = tile_rows<1>(We + (long long)a.N * a.K, a.K, n0, a.N, lane);
  const TileRows<2> w = {{wg.lo[0], wu.lo[0]}, {wg.hi[0], wu.hi[0]}};
  float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
  const bf16* h = a.in + (long long)(lane >> 2) * a.ldin;
  auto x = [&](int k) -> uint4 { return choice >= 0 ? *reinterpret_cast<const uint4*>(h + k) : make_uint4(0, 0, 0, 0); };
  Frag<2, U> cur, nxt;
  load_frag(cur, w, warp * 32, q8, a.K);
  for (int k0 = warp * 32; k0 < a.K; k0 += U * WARPS * 32) {
    if (k0 + U * WARPS * 32 < a.K) load_frag(nxt, w, k0 + U * WARPS * 32, q8, a.K);
    mma_frag(acc, cur, k0, q8, a.K, x);
    cur = nxt;
  }
  spill_tiles<2>(acc, s_acc, warp, lane);
  __syncthreads();
  if (tid < 16 * ROWS) {
    const int m = tid & 15, b = tid >> 4;
    if (s_choice[b] >= 0 && n0 + m < a.N) {
      float g = 0.f, u = 0.f;
#pragma unroll
      for (int i = 0; i < WARPS; ++i) { g += s_acc[i][m][b]; u += s_acc[i][m + 16][b]; }
      a.act[(long long)s_choice[b] * a.N + n0 + m] = __float2bfloat16_rn(g * sigmoidf(g) * u);
    }
  }
}

// grid (ceil(N / 16), CLUSTER), one cluster per 16 outputs: out[b] = mult * sigmoid(g + bias) * sum over the row's experts (+ extra)
__global__ void __cluster_dims__(1, CLUSTER, 1) __launch_bounds__(THREADS)
expert_down_rows_kernel(const ExpertArgs a) {
  constexpr int U = 4;
  __shared__ Choices c;
  __shared__ float s_acc[WARPS][16][ROWS + 1];
  __shared__ float s_part[16][ROWS];
  __shared__ short s_list[MAX_CHOICES];                 // first mentions, in order
  __shared__ short s_pick[ROWS][MAX_CHOICES];           // the row's choice of that expert, or -1
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = a.B * a.top;
  pdl_wait();
  pdl_trigger();
  load_choices(c, a.idx, n);
  for (int i = tid; i < c.distinct * ROWS; i += THREADS) s_pick[i / c.distinct][i % c.distinct] = -1;
  __syncthreads();
  for (int i = tid; i < n; i += THREADS) {
    const int e = c.order[c.first[i]];
    s_pick[i / a.top][e] = (short)i;
    if (c.first[i] == i) s_list[e] = (short)i;
  }
  __syncthreads();
  const int n0 = blockIdx.x * 16, q8 = (lane & 3) * 8, row = lane >> 2;
  float acc[1][4] = {{0.f, 0.f, 0.f, 0.f}};
  // (expert, k) as one loop, the next fragment on its way while the current one is used
  const int per = (a.K + U * WARPS * 32 - 1) / (U * WARPS * 32), rank = blockIdx.y;
  const int steps = per * ((c.distinct - rank + CLUSTER - 1) / CLUSTER);      // experts rank, rank + CLUSTER, ...
  auto fetch = [&](Frag<1, U>& f, int s) {
    const int t = s / per, e = rank + t * CLUSTER, k0 = (s - t * per) * (U * WARPS * 32) + warp * 32;
    load_frag(f, tile_rows<1>(a.W + (long long)c.idx[s_list[e]] * a.N * a.K, a.K, n0, a.N, lane), k0, q8, a.K);
  };
  Frag<1, U> cur, nxt;
  if (steps > 0) fetch(cur, 0);
  for (int s = 0; s < steps; ++s) {
    if (s + 1 < steps) fetch(nxt, s + 1);
    const int t = s / per, e = rank + t * CLUSTER, k0 = (s - t * per) * (U * WARPS * 32) + warp * 32;
    const int choice = row < a.B ? s_pick[row][e] : -1;
    const float wt = choice >= 0 ? a.wt[choice] : 0.f;
    const bf16* in = a.in + (long long)max(choice, 0) * a.K;
    auto x = [&](int k) -> uint4 {
      if (choice < 0) return make_uint4(0, 0, 0, 0);
      float v[8];
      load8(in + k, v);
      return make_uint4(pack_bf16(v[0] * wt, v[1] * wt), pack_bf16(v[2] * wt, v[3] * wt), pack_bf16(v[4] * wt, v[5] * wt), pack_bf16(v[6] * wt, v[7] * wt));
    };
    mma_frag(acc, cur, k0, q8, a.K, x);
    cur = nxt;
  }
  spill_tiles<1>(acc, s_acc, warp, lane);
  __syncthreads();
  const int m = tid & 15, b = tid >> 4, j = n0 + m;
  const float v = cluster_total<16>(s_acc, s_part, tid < 16 * ROWS, m, b);
  if (rank == 0 && tid < 16 * ROWS) {
    if (b < a.B && j < a.N) {
      float r = a.mult * sigmoidf(a.g[b * a.ldg + j] + a.bias[j]) * v;
      if (a.extra) r += a.extra[b * a.ldo + j];
      a.out[b * a.ldo + j] = r;
    }
  }
}

}  // namespace

cudaError_t gemv(const GemvDesc& d, int pre, int epi, cudaStream_t s) {
  if (d.rows < 1 || d.N <= 0 || d.K <= 0 || (d.K & 7) || (d.ldx & 7) || (d.ldw & 7) || d.n_real > d.K) return cudaErrorInvalidValue;
  if (d.rows > ROWS && (pre != PRE_PLAIN || epi == GEMV_RESIDUAL || d.rows > 65535 * ROWS)) return cudaErrorInvalidValue;
  if (pre == PRE_NORM ? (d.w == nullptr || d.n_real <= 0) : (pre != PRE_PLAIN || d.store != nullptr || d.h_out != nullptr)) return cudaErrorInvalidValue;
  if (epi == GEMV_RESIDUAL ? (d.resid == nullptr || d.g == nullptr || d.bias == nullptr) : d.out == nullptr) return cudaErrorInvalidValue;
  if (d.h_out != nullptr && (d.ldh & 7)) return cudaErrorInvalidValue;
  GemvArgs a{};
  a.x = d.x; a.ldx = d.ldx; a.w = d.w; a.eps = d.eps; a.n_real = d.n_real;
  a.W = (const bf16*)d.W; a.ldw = d.ldw; a.B = d.rows; a.N = d.N; a.K = d.K; a.epi = epi; a.accumulate = d.accumulate;
  a.out = d.out; a.ldo = d.ldo; a.resid = d.resid; a.ldr = d.ldr; a.g = d.g; a.ldg = d.ldg; a.bias = d.bias;
  a.mult = d.mult; a.extra = d.extra; a.h_out = (bf16*)d.h_out; a.ldh = d.ldh; a.next = d.next;
  // enough outputs, or groups of rows, for two tiles per CTA: the rows are read half as often
  const bool wide = d.N >= 148 * 32 || (d.rows > ROWS && d.N > 16);
  a.n_blocks = (d.N + (wide ? 31 : 15)) / (wide ? 32 : 16);
  int grid = a.n_blocks;
  if (d.store) { a.store = *d.store; grid += d.rows; }
  if (pre == PRE_PLAIN && !wide && a.n_blocks < 148 && d.K >= 3072 && d.rows <= ROWS) return launch(d.pdl, gemv_cluster_kernel, dim3(grid, CLUSTER), dim3(THREADS), 0, s, a);
  auto kern = pre == PRE_NORM ? (wide ? gemv_kernel<true, 2> : gemv_kernel<true, 1>) : (wide ? gemv_kernel<false, 2> : gemv_kernel<false, 1>);
  return launch(d.pdl, kern, dim3(grid, (d.rows + ROWS - 1) / ROWS), dim3(THREADS), 0, s, a);
}

cudaError_t gemv_relu_glu(const GemvDesc& d, cudaStream_t s) {
  if (d.rows < 1 || d.rows > ROWS || d.N <= 0 || d.K <= 0 || (d.K & 7) || (d.ldx & 7) || (d.ldw & 7) || d.out == nullptr) return cudaErrorInvalidValue;
  GemvArgs a{};
  a.x = d.x; a.ldx = d.ldx; a.W = (const bf16*)d.W; a.ldw = d.ldw; a.B = d.rows; a.N = d.N; a.K = d.K; a.out = d.out; a.ldo = d.ldo; a.next = d.next;
  a.n_blocks = (d.N + 15) / 16;
  return launch(d.pdl, gemv_relu_glu_kernel, dim3(a.n_blocks), dim3(THREADS), 0, s, a);
}

bool expert_rows_supported(int rows, int top) { return rows >= 1 && rows <= ROWS && rows * top <= MAX_CHOICES; }

cudaError_t expert_rows(const ExpertRows& d, cudaStream_t s) {
  if (!expert_rows_supported(d.rows, d.top) || d.top > d.experts || d.K <= 0 || (d.K & 7) || d.fp <= 0 || (d.fp & 7) || d.N <= 0 || (d.ldh & 7) ||
      !d.g || !d.bias || !d.out)
    return cudaErrorInvalidValue;
  ExpertArgs a{};
  a.in = (const bf16*)d.h; a.ldin = d.ldh; a.B = d.rows; a.top = d.top; a.K = d.K; a.N = d.fp; a.W = (const bf16*)d.Wgu; a.idx = d.idx; a.wt = d.wt;
  a.act = (bf16*)d.act;
  const int most = d.rows * d.top < d.experts ? d.rows * d.top : d.experts;
  cudaError_t e = launch(true, expert_gate_up_rows_kernel, dim3(most, (d.fp + 15) / 16), dim3(THREADS), 0, s, a);
  if (e != cudaSuccess) return e;
  a.in = (const bf16*)d.act; a.K = d.fp; a.N = d.N; a.W = (const bf16*)d.Wdown;
  a.out = d.out; a.ldo = d.ldo; a.g = d.g; a.ldg = d.ldg; a.bias = d.bias; a.mult = d.mult; a.extra = d.extra;
  return launch(true, expert_down_rows_kernel, dim3((d.N + 15) / 16, CLUSTER), dim3(THREADS), 0, s, a);
}

}  // namespace serve
}  // namespace nc
