// Mixture of experts.
//
//   moe_route / moe_place   sigmoid or softmax scores, the choice among the best groups, and the (token, choice) pairs laid out expert
//                           after expert
//   moe_gemm (MOE_GLU)      silu(W_gate h) * (W_up h), or its clamped form, over every expert's rows, h gathered by token
//   moe_gemm (MOE_DOWN)     W_down of those rows
//   moe_gemm (ROWS_GLU)     the first product over rows that are in order already
//   moe_norm_add            the weighted sum of a token's rows, a gated shared expert, the norm of the sum, the residual
//
// The products are persistent tcgen05 kernels over the list of (expert, 128-row tile, column tile): TMA brings the weights (one 3-D
// map over all experts, so that a tile past an expert's last row is filled with zeros instead of its neighbour's rows), fp32
// accumulators stay in TMEM, double-buffered.  The GLU form holds gate and up columns of a tile side by side in one accumulator, so
// the activation happens on the way out.  With few rows per expert its token rows are gathered by TMA, four rows a copy; that copy's
// rate would bound the product over long prompts, so there the rows are laid out expert after expert first (moe_gather).  How many rows each expert has is known on the device only: every CTA works out the tile list from the offsets.
#include "host.h"
#include "mma_split.cuh"
#include "vec.cuh"

namespace b2 {

constexpr int MOE_MAX_EXPERTS = 1024;
constexpr int MOE_MAX_TOP = 32;
typedef __nv_bfloat16 moe_bf16;

// ---- routing -----------------------------------------------------------------------------------------------------------
enum : int { SCORE_SIGMOID = 0, SCORE_SOFTMAX = 1 };
struct RouteParams {
  const void* corr;      // T [E] or null
  float* weights;        // [M, slots]
  int* id;               // [M, slots]
  int M, E, top, groups, keep;
  int slots;             // top, or one more: expert E, which every token takes behind a gate of its own
  float scale;
  int score;             // SCORE_*; softmax over all experts
};

// largest value and, among equals, the lowest index
__device__ __forceinline__ void argmax_warp(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float v2 = __shfl_xor_sync(0xffffffffu, v, o);
    const int i2 = __shfl_xor_sync(0xffffffffu, i, o);
    if (v2 > v || (v2 == v && i2 < i)) {
      v = v2;
      i = i2;
    }
  }
}

// The choice of one token by a warp.  z: its logits; sg: the logit of the gate (slots > top); c, gs: E floats of shared memory each
// (choice and group scores).
template <typename T>
__device__ __forceinline__ void route_token(const RouteParams& p, int row, const float* z, const float* sg, float* c, float* gs) {
  const int lane = threadIdx.x & 31;
  constexpr float LOW = -3.0e38f;           // in place of what is no number (rows without a sequence): below any score, above "closed"
  float most = -INFINITY, total = 0.f;
  if (p.score == SCORE_SOFTMAX) {
    for (int e = lane; e < p.E; e += 32) most = fmaxf(most, z[e]);
    most = warp_max(most);
    for (int e = lane; e < p.E; e += 32) total += expf(z[e] - most);
    total = warp_sum(total);
  }
  auto score = [&](float v) { return p.score == SCORE_SOFTMAX ? expf(v - most) / total : sigmoid_f(v); };
  const bool by_logit = p.corr == nullptr && p.keep == p.groups;      // the order of the scores is that of the logits
  for (int e = lane; e < p.E; e += 32) {
    const float s = by_logit ? z[e] : score(z[e]) + (p.corr ? to_f(static_cast<const T*>(p.corr)[e]) : 0.f);
    c[e] = s >= LOW ? s : LOW;
  }
  __syncwarp();
  const int per = p.E / p.groups;
  const bool narrow = p.E <= 4 * 32;        // few enough to find every expert's rank by comparing it with all others
  if (p.keep < p.groups) {
    for (int g = lane; g < p.groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const float v = c[e];
        b = fmaxf(b, fminf(a, v));
        a = fmaxf(a, v);
      }
      gs[g] = per > 1 ? fmaxf(a + b, LOW) : a;
    }
    __syncwarp();
    if (narrow) {
      float mine[4];                        // +inf for a kept group, -inf for a closed one
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int g = lane + 32 * j;
        if (g >= p.groups) break;
        const float v = gs[g];
        int rank = 0;
        for (int o = 0; o < p.groups; ++o) {
          const float w = gs[o];
          rank += w > v || (w == v && o < g);
        }
        mine[j] = rank < p.keep ? INFINITY : -INFINITY;
      }
      __syncwarp();
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (lane + 32 * j < p.groups) gs[lane + 32 * j] = mine[j];
      __syncwarp();
    } else {
      for (int k = 0; k < p.keep; ++k) {    // a kept group's score becomes +inf
        float v = -INFINITY;
        int at = p.groups;
        for (int g = lane; g < p.groups; g += 32)
          if (gs[g] > v && gs[g] != INFINITY) {
            v = gs[g];
            at = g;
          }
        argmax_warp(v, at);
        if (lane == 0 && at < p.groups) gs[at] = INFINITY;
        __syncwarp();
      }
    }
    for (int e = lane; e < p.E; e += 32)
      if (gs[e / per] != INFINITY) c[e] = -INFINITY;
    __syncwarp();
  }
  const size_t first = static_cast<size_t>(row) * p.slots;
  auto choose = [&](int k, int e) {
    p.weights[first + k] = score(z[e]) * p.scale;
    p.id[first + k] = e;
  };
  if (p.slots > p.top && lane == 31) {
    p.weights[first + p.top] = sigmoid_f(*sg);
    p.id[first + p.top] = p.E;
  }
  if (narrow) {
    for (int e = lane; e < p.E; e += 32) {
      const float v = c[e];
      int rank = 0;
      for (int o = 0; o < p.E; ++o) {
        const float w = c[o];
        rank += w > v || (w == v && o < e);
      }
      if (rank < p.top) choose(rank, e);
    }
  } else {
    int mine = 0;
    for (int k = 0; k < p.top; ++k) {
      float v = -INFINITY;
      int at = p.E;
      for (int e = lane; e < p.E; e += 32)
        if (c[e] > v) {
          v = c[e];
          at = e;
        }
      argmax_warp(v, at);
      at = min(at, p.E - 1);
      if (lane == k) mine = at;
      if (lane == 0) c[at] = -INFINITY;
      __syncwarp();
    }
    if (lane < p.top) choose(lane, mine);
  }
  __syncwarp();
}

// Logits given: a warp per token.
constexpr int MR_WARPS = 4;
template <typename T>
__global__ void __launch_bounds__(MR_WARPS * 32) moe_route_kernel(const RouteParams p, const float* __restrict__ z, long long ld,
                                                                   const float* __restrict__ sg, long long ld_sg) {
  extern __shared__ float mr_smem[];
  const int warp = threadIdx.x >> 5, row = blockIdx.x * MR_WARPS + warp;
  if (row >= p.M) return;
  float* c = mr_smem + warp * 2 * p.E;
  route_token<T>(p, row, z + static_cast<size_t>(row) * ld, sg + static_cast<size_t>(row) * ld_sg, c, c + p.E);
}

// Products with few outputs or few rows (router logits, gates), bf16 operands and a 32-bit result: 16 rows and up to 72 columns a CTA,
// whose warps split the contraction.  A lane loads eight neighbouring elements of its row of either operand at once and uses them as
// the fragments of two m16n8k16 products: the order of the contraction is free as long as both operands agree on it.  SK_ROUTE: the rows' experts are chosen on the
// spot.  SK_TOKEN: the result goes through gelu and times a vector of the row's token, rounded to bf16.
enum : int { SK_PLAIN = 0, SK_ROUTE = 1, SK_TOKEN = 2 };
struct SkinnyParams {
  const moe_bf16* h;     // [M, ld_h]
  const moe_bf16* w;     // [N, ld_w]
  float* z;              // [M, ld_z]; ROUTE: only column sg is stored, if at all (null, or sg < 0)
  long long ld_h, ld_w, ld_z;
  int M, N, K, sg;
  const moe_bf16* table; // SK_TOKEN: [vocab, ld_table], columns first .. first + N - 1
  const long long* ids;  // [M]
  moe_bf16* out;         // [M, N]
  long long ld_table;
  int first, vocab;
};
constexpr int SK_ROWS = 16, SK_WARPS = 8, SK_MAX_TILES = 9;

template <int NT, int FORM>
__global__ void __launch_bounds__(SK_WARPS * 32) skinny_kernel(const SkinnyParams p, const RouteParams r) {
  constexpr int NP = NT * 8, LD = NP + 2;
  constexpr bool ROUTE = FORM == SK_ROUTE;
  const int n0 = blockIdx.y * NP;
  __shared__ float part[SK_WARPS][SK_ROWS][LD];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3, m0 = blockIdx.x * SK_ROWS;
  const moe_bf16* a0 = p.h + static_cast<size_t>(min(m0 + g, p.M - 1)) * p.ld_h;
  const moe_bf16* a1 = p.h + static_cast<size_t>(min(m0 + g + 8, p.M - 1)) * p.ld_h;
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
  constexpr int U = NT <= 2 ? 8 : NT <= 5 ? 4 : 2;        // steps whose loads are in flight together
  const uint4 zero = make_uint4(0, 0, 0, 0);
  for (int k0 = warp * 32; k0 < p.K; k0 += U * SK_WARPS * 32) {
    uint4 x0[U], x1[U], w[U][NT];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = k0 + u * (SK_WARPS * 32) + t * 8;
      const bool in = k < p.K;               // p.K is a multiple of 8
      x0[u] = in ? *reinterpret_cast<const uint4*>(a0 + k) : zero;
      x1[u] = in ? *reinterpret_cast<const uint4*>(a1 + k) : zero;
#pragma unroll
      for (int n = 0; n < NT; ++n)
        w[u][n] = in && n0 + n * 8 + g < p.N ? *reinterpret_cast<const uint4*>(p.w + static_cast<size_t>(n0 + n * 8 + g) * p.ld_w + k) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t f0[4] = {x0[u].x, x1[u].x, x0[u].y, x1[u].y}, f1[4] = {x0[u].z, x1[u].z, x0[u].w, x1[u].w};
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const uint32_t b0[2] = {w[u][n].x, w[u][n].y}, b1[2] = {w[u][n].z, w[u][n].w};
        mma_bf16(acc[n], f0, b0);
        mma_bf16(acc[n], f1, b1);
      }
    }
  }
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    *reinterpret_cast<float2*>(&part[warp][g][n * 8 + 2 * t]) = make_float2(acc[n][0], acc[n][1]);
    *reinterpret_cast<float2*>(&part[warp][g + 8][n * 8 + 2 * t]) = make_float2(acc[n][2], acc[n][3]);
  }
  __syncthreads();
  for (int i = tid; i < SK_ROWS * NP; i += SK_WARPS * 32) {
    const int row = i / NP, c = i % NP;
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < SK_WARPS; ++w) s += part[w][row][c];
    if (ROUTE) part[0][row][c] = s;          // read by this thread alone until the barrier
    if (FORM == SK_TOKEN) {
      if (m0 + row < p.M && n0 + c < p.N) {
        const long long id = p.ids[m0 + row];
        const float t = id >= 0 && id < p.vocab ? to_f(p.table[id * p.ld_table + p.first + n0 + c]) : 0.f;
        p.out[static_cast<size_t>(m0 + row) * p.N + n0 + c] = from_f<moe_bf16>(gelu_tanh_t<moe_bf16>(s) * t);
      }
      continue;
    }
    if (m0 + row < p.M && (ROUTE ? c == p.sg && p.z != nullptr : n0 + c < p.N)) p.z[static_cast<size_t>(m0 + row) * p.ld_z + (ROUTE ? 0 : n0 + c)] = s;
  }
  if (!ROUTE) return;
  __syncthreads();
  for (int row = warp; row < SK_ROWS && m0 + row < p.M; row += SK_WARPS)
    route_token<moe_bf16>(r, m0 + row, part[0][row], &part[0][row][max(p.sg, 0)], part[1 + (warp >> 1)][(warp & 1) * 8],
                          part[1 + (warp >> 1)][(warp & 1) * 8 + 1]);
}

// Running sums of f(i) over i < n by a whole warp: out[0 .. n].
template <typename F>
__device__ __forceinline__ void warp_prefix(int n, int* out, F f) {
  const int lane = threadIdx.x & 31;
  int carry = 0;
  for (int i0 = 0; i0 < n; i0 += 32) {
    const int i = i0 + lane;
    int v = i < n ? f(i) : 0;
    const int own = v;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int t = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += t;
    }
    if (i < n) out[i] = carry + v - own;
    carry += __shfl_sync(0xffffffffu, v, 31);
  }
  if (lane == 0) out[n] = carry;
}

// An index that came from memory and is outside its range: recorded, and the access left out.
__device__ __forceinline__ bool moe_bad(bool bad, int* status) {
  if (bad) atomicCAS(status, 0, ERR_BAD_ARGUMENT);
  return bad;
}

// The layout of the (token, choice) pairs.  Up to MP_ONE pairs: one CTA counts in shared memory.
constexpr int MP_THREADS = 1024, MP_EACH = 16, MP_ONE = MP_THREADS * MP_EACH;
__global__ void __launch_bounds__(MP_THREADS) moe_place_kernel(const int* __restrict__ id, int* __restrict__ place, int* __restrict__ token,
                                                               int* __restrict__ offsets, int E, int top, int total, int* status) {
  __shared__ int cnt[MOE_MAX_EXPERTS], off[MOE_MAX_EXPERTS + 1];
  for (int e = threadIdx.x; e < E; e += MP_THREADS) cnt[e] = 0;
  __syncthreads();
  int e[MP_EACH], rank[MP_EACH];
#pragma unroll
  for (int j = 0; j < MP_EACH; ++j) {
    const int i = threadIdx.x + j * MP_THREADS;
    e[j] = i < total ? id[i] : 0;
    if (moe_bad(e[j] < 0 || e[j] >= E, status)) e[j] = 0;
  }
#pragma unroll
  for (int j = 0; j < MP_EACH; ++j)
    if (static_cast<int>(threadIdx.x) + j * MP_THREADS < total) rank[j] = atomicAdd(cnt + e[j], 1);
  __syncthreads();
  if (threadIdx.x < 32) warp_prefix(E, off, [&](int k) { return cnt[k]; });
  __syncthreads();
  for (int k = threadIdx.x; k <= E; k += MP_THREADS) offsets[k] = off[k];
#pragma unroll
  for (int j = 0; j < MP_EACH; ++j) {
    const int i = threadIdx.x + j * MP_THREADS;
    if (i >= total) break;
    const int r = off[e[j]] + rank[j];
    place[i] = r;
    token[r] = i / top;
  }
}

// More pairs: every CTA counts its own, takes its places among the experts' rows (count, zero before), then the same once the counts
// are complete.
__global__ void __launch_bounds__(256) moe_rank_kernel(int* __restrict__ id, int* __restrict__ place, int* __restrict__ count, int E,
                                                       int total, int* status) {
  __shared__ int cnt[MOE_MAX_EXPERTS];
  for (int e = threadIdx.x; e < E; e += 256) cnt[e] = 0;
  __syncthreads();
  int e[4], rank[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int i = (blockIdx.x * 4 + j) * 256 + threadIdx.x;
    if (i < total) {
      e[j] = id[i];
      if (moe_bad(e[j] < 0 || e[j] >= E, status)) id[i] = e[j] = 0;
      rank[j] = atomicAdd(cnt + e[j], 1);
    }
  }
  __syncthreads();
  for (int k = threadIdx.x; k < E; k += 256)
    if (cnt[k] > 0) cnt[k] = atomicAdd(count + k, cnt[k]);
  __syncthreads();
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int i = (blockIdx.x * 4 + j) * 256 + threadIdx.x;
    if (i < total) place[i] = cnt[e[j]] + rank[j];
  }
}
__global__ void __launch_bounds__(256) moe_layout_kernel(const int* __restrict__ count, const int* __restrict__ id, int* __restrict__ place,
                                                         int* __restrict__ token, int* __restrict__ offsets, int E, int top, int total,
                                                         int* status) {
  __shared__ int off[MOE_MAX_EXPERTS + 1];
  if (threadIdx.x < 32) warp_prefix(E, off, [&](int e) { return count[e]; });
  __syncthreads();
  if (blockIdx.x == 0)
    for (int e = threadIdx.x; e <= E; e += 256) offsets[e] = off[e];
  for (int i = blockIdx.x * 256 + threadIdx.x; i < total; i += gridDim.x * 256) {
    int r = off[id[i]] + place[i];
    if (moe_bad(r < 0 || r >= total, status)) r = 0;
    place[i] = r;
    token[r] = i / top;
  }
}

// ---- grouped products ----------------------------------------------------------------------------------------------------
// The tile list: expert e has ceil(rows / tile) row tiles, first[e] of them before it.
struct MoeTile {
  int expert, row0, rows, col;       // rows of the layout; column tile
};
__device__ __forceinline__ MoeTile moe_tile(int t, const int* off, const int* first, int E, int tile, int ncols) {
  // tiles of one expert are neighbours, its row tiles innermost: they share the weights' columns
  int lo = 0, hi = E;
  while (hi - lo > 1) {
    const int mid = (lo + hi) / 2;
    if (first[mid] * ncols <= t) lo = mid;
    else hi = mid;
  }
  const int n = first[lo + 1] - first[lo], in = t - first[lo] * ncols;
  MoeTile r;
  r.expert = lo;
  r.col = in / n;
  r.row0 = off[lo] + in % n * tile;
  r.rows = min(tile, off[lo + 1] - r.row0);
  return r;
}

// What a gated product does with gate and up: silu(g) u, or with g = min(g, limit), u = clamp(u, -limit, limit): g sigmoid(alpha g) (u + 1)
enum : int { GLU_SILU = 0, GLU_CLAMPED = 1 };
struct GluAct {
  int kind;
  float alpha, limit;
};
__device__ __forceinline__ float clamped_glu(float g, float u, const GluAct& a) {
  g = fminf(g, a.limit);
  u = fminf(fmaxf(u, -a.limit), a.limit);
  return g * sigmoid_f(a.alpha * g) * (u + 1.f);
}
// two values with one reciprocal between them, for results that are rounded to bf16 next
__device__ __forceinline__ void clamped_glu_pair_fast(float& g0, float& g1, float u0, float u1, const GluAct& a) {
  g0 = fminf(g0, a.limit);
  g1 = fminf(g1, a.limit);
  u0 = fminf(fmaxf(u0, -a.limit), a.limit);
  u1 = fminf(fmaxf(u1, -a.limit), a.limit);
  const float k = -1.4426950408889634f * a.alpha;
  const float d0 = 1.f + fast_exp2(fminf(k * g0, 62.f)), d1 = 1.f + fast_exp2(fminf(k * g1, 62.f));
  const float r = __fdividef(1.f, d0 * d1);
  g0 *= r * d1 * (u0 + 1.f);
  g1 *= r * d0 * (u1 + 1.f);
}

// 32-bit form: 64 x 64 tiles of plain FMAs.  Grid (column tiles, an upper bound of the row tiles).
constexpr int MF_T = 64, MF_K = 16;
template <bool GLU>
__global__ void __launch_bounds__(256) moe_gemm_f32_kernel(const float* __restrict__ A, long long lda, const float* __restrict__ W,
                                                           const int* __restrict__ token, const int* __restrict__ offsets,
                                                           float* __restrict__ out, int E, int N, int K, const GluAct act) {
  __shared__ int off[MOE_MAX_EXPERTS + 1], first[MOE_MAX_EXPERTS + 1];
  __shared__ __align__(16) float sA[MF_K][MF_T + 4], sB[GLU ? 2 : 1][MF_K][MF_T + 4];   // read in vectors of four
  for (int e = threadIdx.x; e <= E; e += 256) off[e] = offsets[e];
  __syncthreads();
  if (threadIdx.x < 32) warp_prefix(E, first, [&](int e) { return (off[e + 1] - off[e] + MF_T - 1) / MF_T; });
  __syncthreads();
  if (static_cast<int>(blockIdx.y) >= first[E]) return;
  const MoeTile tl = moe_tile(blockIdx.y, off, first, E, MF_T, 1);
  const int n0 = blockIdx.x * MF_T, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const float* w = W + static_cast<size_t>(tl.expert) * (GLU ? 2 : 1) * N * K;
  float acc[GLU ? 2 : 1][4][4] = {};
  for (int k0 = 0; k0 < K; k0 += MF_K) {
    for (int i = threadIdx.x; i < MF_T * MF_K; i += 256) {
      const int r = i / MF_K, k = i % MF_K;
      const bool in = k0 + k < K;
      const size_t row = GLU ? (r < tl.rows ? token[tl.row0 + r] : 0) : tl.row0 + r;
      sA[k][r] = in && r < tl.rows ? A[row * lda + k0 + k] : 0.f;
#pragma unroll
      for (int g = 0; g < (GLU ? 2 : 1); ++g)
        sB[g][k][r] = in && n0 + r < N ? w[(static_cast<size_t>(g) * N + n0 + r) * K + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < MF_K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sA[k][ty * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
      for (int g = 0; g < (GLU ? 2 : 1); ++g) {
        const float4 b = *reinterpret_cast<const float4*>(&sB[g][k][tx * 4]);
        const float bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[g][i][j] = fmaf(av[i], bv[j], acc[g][i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = ty * 4 + i;
    if (m >= tl.rows) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      const float g = acc[0][i][j], u = acc[GLU ? 1 : 0][i][j];
      out[static_cast<size_t>(tl.row0 + m) * N + n] = !GLU ? g : act.kind == GLU_CLAMPED ? clamped_glu(g, u, act) : silu_f(g) * u;
    }
  }
}

constexpr int MG_BM = 128, MG_BK = 64;
template <int BN>
struct MoeCfg {
  static constexpr int A_BYTES = MG_BM * MG_BK * 2, B_BYTES = BN * MG_BK * 2, STAGE = A_BYTES + B_BYTES;
  static constexpr int STAGES = BN == 256 ? 4 : BN == 128 ? 6 : 8;
  static constexpr int STAGING = 4 * 4096;                        // a block per epilogue warp
  static constexpr int TABLES = 2 * (MOE_MAX_EXPERTS + 1) * 4;
  static constexpr int SMEM = STAGES * STAGE + STAGING + 256 + TABLES + 1024;
  static constexpr int TMEM = 2 * BN;
};

enum : int { MOE_GLU = 0, MOE_DOWN = 1, ROWS_GLU = 2 };

struct MoeGemmParams {
  const int* token;        // MOE_GLU: [P]
  const int* offsets;      // [E + 1], or null: one expert, all rows
  moe_bf16* out;           // [P, ld_out]
  long long ld_out;
  int P, E, N, K;          // GLU: N activation columns (half of a tile's accumulator columns each for gate and up)
  GluAct act;
};

template <int BN, int FORM>
__global__ void __launch_bounds__(192, 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB, const MoeGemmParams p, int* status) {
  using Cfg = MoeCfg<BN>;
  constexpr bool GLU = FORM != MOE_DOWN;
  constexpr int STAGES = Cfg::STAGES, COLS = GLU ? BN / 2 : BN;    // output columns of a tile
  extern __shared__ uint8_t mg_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(mg_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t* staging = smem + STAGES * Cfg::STAGE;
  uint64_t* full = reinterpret_cast<uint64_t*>(staging + Cfg::STAGING);
  uint64_t *empty = full + STAGES, *acc_full = empty + STAGES, *acc_empty = acc_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
  int* off = reinterpret_cast<int*>(staging + Cfg::STAGING + 256);
  int* first = off + MOE_MAX_EXPERTS + 1;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(full + i, 1);
      mbar_init(empty + i, 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(acc_full + i, 1);
      mbar_init(acc_empty + i, 4);
    }
    mbar_fence_init();
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmB);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, Cfg::TMEM);
    tmem_relinquish();
  }
  for (int e = tid; e <= p.E; e += blockDim.x) off[e] = p.offsets ? p.offsets[e] : e * p.P;
  __syncthreads();
  if (warp == 0) warp_prefix(p.E, first, [&](int e) { return (off[e + 1] - off[e] + MG_BM - 1) / MG_BM; });
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(tmem_slot);
  const bool sound = off[0] == 0 && off[p.E] == p.P;           // else nothing is computed
  if (tid == 0) moe_bad(!sound, status);
  const int ncols = (p.N + COLS - 1) / COLS, tiles = sound ? first[p.E] * ncols : 0, nkb = (p.K + MG_BK - 1) / MG_BK;

  if (warp == 0) {
    // Lane l gathers rows 4 l .. 4 l + 3 of a tile; a group that reaches past the expert's last row repeats it, groups further on keep
    // what they hold: those results are dropped.
    int st = 0;
    uint32_t ph = 0;
    bool ok = true;
    for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
      const MoeTile tl = moe_tile(t, off, first, p.E, MG_BM, ncols);
      const int groups = (tl.rows + 3) / 4;
      int y[4] = {};
      if (FORM == MOE_GLU && lane < groups)
#pragma unroll
        for (int i = 0; i < 4; ++i) y[i] = p.token[tl.row0 + min(lane * 4 + i, tl.rows - 1)];
      for (int kb = 0; kb < nkb; ++kb) {
        if (!mbar_wait_warp(empty + st, ph ^ 1, status, ERR_GEMM_PRODUCER_WAIT)) {
          ok = false;
          break;
        }
        uint8_t *sA = smem + st * Cfg::STAGE, *sB = sA + Cfg::A_BYTES;
        if (lane == 0) {
          mbar_expect_tx(full + st, Cfg::B_BYTES + (FORM == MOE_GLU ? groups * 512 : Cfg::A_BYTES));
          if (GLU) {
            tma_load_3d(sB, &tmB, full + st, kb * MG_BK, tl.col * COLS, 2 * tl.expert);
            tma_load_3d(sB + Cfg::B_BYTES / 2, &tmB, full + st, kb * MG_BK, tl.col * COLS, 2 * tl.expert + 1);
          } else {
            tma_load_3d(sB, &tmB, full + st, kb * MG_BK, tl.col * COLS, tl.expert);
          }
          if (FORM != MOE_GLU) tma_load_2d(sA, &tmA, full + st, kb * MG_BK, tl.row0);
        }
        __syncwarp();
        if (FORM == MOE_GLU && lane < groups) tma_gather4(sA + lane * 512, &tmA, full + st, kb * MG_BK, y[0], y[1], y[2], y[3]);
        if (++st == STAGES) {
          st = 0;
          ph ^= 1;
        }
      }
    }
  } else if (warp == 1) {
    const bool leader = elect_one();
    constexpr uint32_t idesc = make_idesc_f16(1, MG_BM, BN, 0, 0);
    int st = 0, acc = 0;
    uint32_t ph = 0, acc_ph = 0;
    bool ok = true;
    for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
      if (!mbar_wait(acc_empty + acc, acc_ph ^ 1, status, ERR_GEMM_MMA_WAIT_TMEM)) break;
      tc_fence_after();
      for (int kb = 0; kb < nkb; ++kb) {
        if (!mbar_wait(full + st, ph, status, ERR_GEMM_MMA_WAIT_FULL)) {
          ok = false;
          break;
        }
        tc_fence_after();
        const uint32_t a_base = smem_u32(smem + st * Cfg::STAGE);
        const uint64_t a0 = make_smem_desc_sw128(a_base, 16, 1024), b0 = make_smem_desc_sw128(a_base + Cfg::A_BYTES, 16, 1024);
        if (leader) {
#pragma unroll
          for (int k = 0; k < MG_BK / 16; ++k)
            umma_f16_ss(tmem + acc * BN, desc_advance(a0, k * 32), desc_advance(b0, k * 32), idesc, kb > 0 || k > 0 ? 1u : 0u);
          umma_commit(empty + st);
        }
        if (++st == STAGES) {
          st = 0;
          ph ^= 1;
        }
      }
      if (!ok) break;
      if (leader) umma_commit(acc_full + acc);
      acc ^= 1;
      if (acc == 0) acc_ph ^= 1;
    }
  } else {
    const int quarter = warp & 3;
    uint8_t* stage = staging + quarter * 4096;
    int acc = 0;
    uint32_t acc_ph = 0;
    for (int t = blockIdx.x; t < tiles; t += gridDim.x) {
      const MoeTile tl = moe_tile(t, off, first, p.E, MG_BM, ncols);
      if (!mbar_wait_warp(acc_full + acc, acc_ph, status, ERR_GEMM_EPI_WAIT)) break;
      tc_fence_after();
      const uint32_t at = tmem + (static_cast<uint32_t>(quarter * 32) << 16) + acc * BN;
      const bool live = quarter * 32 < tl.rows;
#pragma unroll 1
      for (int c0 = 0; c0 < COLS; c0 += 64) {
        if (!live || tl.col * COLS + c0 >= p.N) break;
        uint4 v[8];
        constexpr int W32 = COLS < 64 ? COLS / 32 : 2;
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          uint32_t r[32];
          if (hh >= W32) {
#pragma unroll
            for (int j = 0; j < 4; ++j) v[hh * 4 + j] = make_uint4(0, 0, 0, 0);
            continue;
          }
          tmem_ld_32x32b_x32(at + c0 + hh * 32, r);
          if (GLU) {
            uint32_t u[32];
            tmem_ld_32x32b_x32(at + BN / 2 + c0 + hh * 32, u);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              float x = __uint_as_float(r[i]), y = __uint_as_float(r[i + 1]);
              if (p.act.kind == GLU_CLAMPED) {
                clamped_glu_pair_fast(x, y, __uint_as_float(u[i]), __uint_as_float(u[i + 1]), p.act);
              } else {
                silu_pair_fast(x, y);
                x *= __uint_as_float(u[i]);
                y *= __uint_as_float(u[i + 1]);
              }
              r[i] = __float_as_uint(x);
              r[i + 1] = __float_as_uint(y);
            }
          } else {
            tmem_ld_wait();
          }
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            uint32_t o[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) o[e] = pack_bf16x2(__uint_as_float(r[8 * j + 2 * e]), __uint_as_float(r[8 * j + 2 * e + 1]));
            v[hh * 4 + j] = make_uint4(o[0], o[1], o[2], o[3]);
          }
        }
        const int col = tl.col * COLS + c0;
        moe_bf16* base = p.out + static_cast<size_t>(tl.row0 + quarter * 32) * p.ld_out + col;
        warp_store_rows_128B(stage, v, [&](int row) -> uint8_t* {
          if (quarter * 32 + row >= tl.rows || col + (lane & 7) * 8 >= p.N || c0 + (lane & 7) * 8 >= COLS) return nullptr;
          return reinterpret_cast<uint8_t*>(base + static_cast<size_t>(row) * p.ld_out);
        });
      }
      tc_fence_before();
      mbar_arrive_warp(acc_empty + acc);
      acc ^= 1;
      if (acc == 0) acc_ph ^= 1;
    }
  }
  if (*reinterpret_cast<volatile int*>(status) != 0) {     // copies and products in flight land before shared memory and TMEM go away
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::TMEM);
  }
}

// rows[r] = h[token[r]], a warp per row (16 bytes a lane)
__global__ void __launch_bounds__(256) moe_gather_kernel(const moe_bf16* __restrict__ h, long long ld, const int* __restrict__ token,
                                                         moe_bf16* __restrict__ rows, int tokens, int P, int K, int* status) {
  for (int r = blockIdx.x * 8 + (threadIdx.x >> 5); r < P; r += gridDim.x * 8) {
    const int from = token[r];
    if (moe_bad(from < 0 || from >= tokens, status)) continue;
    const uint4* src = reinterpret_cast<const uint4*>(h + static_cast<size_t>(from) * ld);
    uint4* dst = reinterpret_cast<uint4*>(rows + static_cast<size_t>(r) * K);
    const int n = K / 8;
    for (int c0 = threadIdx.x & 31; c0 < n; c0 += 128) {
      uint4 v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (c0 + 32 * i < n) v[i] = src[c0 + 32 * i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (c0 + 32 * i < n) dst[c0 + 32 * i] = v[i];
    }
  }
}

// ---- weighted sum, norm, residual ---------------------------------------------------------------------------------------------
struct MoeAddParams {
  float* x;              // [M, ld]
  const void* rows;      // T [P, ld]
  const int* place;      // [M, top]
  const float* weights;  // [M, top]
  const float* shared;   // [M, ld] or null
  const float* sg;       // [M], stride ld_sg: gate before its sigmoid
  const void* w;         // T [ld]
  void* h;               // T [M, ld] or null
  int top, P, ld_sg, ld, n;
  float coef, eps;
  int* status;
};

__device__ __forceinline__ float moe_block_sum(float v, float* scratch) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  const int lane = threadIdx.x & 31;
  return warp_sum(lane < static_cast<int>(blockDim.x >> 5) ? scratch[lane] : 0.f);
}

template <typename T, int V, int MAXT>
__global__ void __launch_bounds__(MAXT) moe_norm_add_kernel(const MoeAddParams p) {
  __shared__ float scratch[32], sw[MOE_MAX_TOP];
  __shared__ int sr[MOE_MAX_TOP];
  const size_t base = static_cast<size_t>(blockIdx.x) * p.ld;
  if (static_cast<int>(threadIdx.x) < p.top) {
    sw[threadIdx.x] = p.weights[static_cast<size_t>(blockIdx.x) * p.top + threadIdx.x];
    const int r = p.place[static_cast<size_t>(blockIdx.x) * p.top + threadIdx.x];
    sr[threadIdx.x] = moe_bad(r < 0 || r >= p.P, p.status) ? 0 : r;
  }
  const float g = p.shared ? sigmoid_f(p.sg[static_cast<size_t>(blockIdx.x) * p.ld_sg]) : 0.f;
  __syncthreads();
  const T* rows = static_cast<const T*>(p.rows);
  float a[V][8], b[V][8], ss = 0.f;
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
#pragma unroll
    for (int e = 0; e < 8; ++e) a[k][e] = b[k][e] = 0.f;
    if (c >= p.ld) continue;
    vload8(p.x + base + c, b[k]);
    if (p.shared) {
      vload8(p.shared + base + c, a[k]);
#pragma unroll
      for (int e = 0; e < 8; ++e) a[k][e] *= g;
    }
    for (int j = 0; j < p.top; j += 4) {
      float t[4][8];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (j + i < p.top) vload8(rows + static_cast<size_t>(sr[j + i]) * p.ld + c, t[i]);
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (j + i < p.top)
#pragma unroll
          for (int e = 0; e < 8; ++e) a[k][e] = fmaf(sw[j + i], t[i][e], a[k][e]);
    }
  }
#pragma unroll
  for (int k = 0; k < V; ++k)
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(a[k][e], a[k][e], ss);
  const float r = p.coef / sqrtf(moe_block_sum(ss, scratch) / p.n + p.eps);
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c >= p.ld) break;
    float wv[8];
    vload8(static_cast<const T*>(p.w) + c, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) b[k][e] = fmaf(a[k][e] * r, wv[e], b[k][e]);
    vstore8(p.x + base + c, b[k]);
    if (p.h) vstore8(static_cast<T*>(p.h) + base + c, b[k]);
  }
}

template <int BN, int FORM>
static int launch_moe(const CUtensorMap* ta, const CUtensorMap* tb, const MoeGemmParams& p, int bound, cudaStream_t stream) {
  using Cfg = MoeCfg<BN>;
  auto kern = moe_gemm_kernel<BN, FORM>;
  int* status = status_ptr();
  if (!status) return 3;
  static bool set[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!set[dev & 63]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM) != cudaSuccess) {
      set_error("moe_gemm: cannot set shared memory size (%d)", Cfg::SMEM);
      return 1;
    }
    set[dev & 63] = true;
  }
  constexpr int COLS = FORM != MOE_DOWN ? BN / 2 : BN;
  const long long tiles = static_cast<long long>(bound) * ((p.N + COLS - 1) / COLS);
  const int grid = tiles < num_sms() ? static_cast<int>(tiles) : num_sms();
  kern<<<grid, 192, Cfg::SMEM, stream>>>(*ta, *tb, p, status);
  B2_CHECK_LAUNCH("moe_gemm");
  return 0;
}

// Gate and up [E, 2, F, K] in tiles of `cols` activation columns.
template <int FORM>
static int launch_glu(const CUtensorMap* ta, const void* w, const MoeGemmParams& p, int cols, int bound, cudaStream_t stream) {
  const uint64_t dims[3] = {static_cast<uint64_t>(p.K), static_cast<uint64_t>(p.N), 2ull * p.E},
                 strides[2] = {2ull * p.K, 2ull * p.N * p.K};
  const uint32_t box[3] = {MG_BK, static_cast<uint32_t>(cols), 1};
  const CUtensorMap* tb = tensor_map_nd_bf16(w, 3, dims, strides, box, 3);
  if (!ta || !tb) return 2;
  if (cols == 128) return launch_moe<256, FORM>(ta, tb, p, bound, stream);
  if (cols == 64) return launch_moe<128, FORM>(ta, tb, p, bound, stream);
  return launch_moe<64, FORM>(ta, tb, p, bound, stream);
}

static int moe_bound(int P, int E, int tile) { return P / tile + (E < P ? E : P); }    // row tiles at most

// Column tile: the one whose last wave wastes least, by the expected number of row tiles; a tile costs its columns and a fixed part.
static int moe_columns(int P, int E, int N, int widest, int narrowest) {
  const int used = E < P ? E : P;
  const long long rows = static_cast<long long>(used) * ((P / used + MG_BM - 1) / MG_BM);
  int best = widest;
  long long least = -1;
  for (int cols = widest; cols >= narrowest; cols /= 2) {
    const long long tiles = rows * ((N + cols - 1) / cols), cost = (tiles + num_sms() - 1) / num_sms() * (cols + 32);
    if (least < 0 || cost < least) {
      least = cost;
      best = cols;
    }
  }
  return best;
}

}  // namespace b2

using namespace b2;

static bool bad_routing(int M, int E, int top, int groups, int keep, int slots) {
  if (E < 1 || E + 1 > MOE_MAX_EXPERTS || (slots != top && slots != top + 1) || slots > MOE_MAX_TOP || groups < 1 || E % groups || keep < 1 || keep > groups || top < 1 || top > MOE_MAX_TOP ||
      top > keep * (E / groups) || static_cast<long long>(M) * slots > 0x7fffffffll) {
    set_error("moe_route: fewer than %d experts in equal groups and up to %d chosen required", MOE_MAX_EXPERTS, MOE_MAX_TOP);
    return true;
  }
  return false;
}

// work: [E] counts, then [M * top] chosen experts (both with the expert that every token takes, if there is one)
static int launch_place(int* place, int* token, int* offsets, int* work, int M, int E, int top, cudaStream_t st) {
  const int total = M * top;
  int *id = work + E, *status = status_ptr();
  if (!status) return 3;
  if (total <= MP_ONE) {
    moe_place_kernel<<<1, MP_THREADS, 0, st>>>(id, place, token, offsets, E, top, total, status);
    B2_CHECK_LAUNCH("moe_place");
    return 0;
  }
  if (cudaMemsetAsync(work, 0, sizeof(int) * E, st) != cudaSuccess) { set_error("moe_place: clearing the counts failed"); return 5; }
  moe_rank_kernel<<<(total + 1023) / 1024, 256, 0, st>>>(id, place, work, E, total, status);
  B2_CHECK_LAUNCH("moe_rank");
  moe_layout_kernel<<<2 * num_sms(), 256, 0, st>>>(work, id, place, token, offsets, E, top, total, status);
  B2_CHECK_LAUNCH("moe_layout");
  return 0;
}

// z: fp32 [M, ld]; work: int32 [E + M * top]; offsets: int32 [E + 1]; place: int32 [M, top]; token: int32 [M * top].  joint: every token
// also takes expert E, with the weight sigmoid(sg) (fp32 [M], stride ld_sg); then one more expert and choice in all of these.  softmax:
// scores are a softmax over all experts instead of a sigmoid each; corr may be null.
B2_EXPORT int b2_moe_route(const float* z, long long ld, const float* sg, long long ld_sg, int joint, const void* corr, float* weights,
                           int* place, int* token, int* offsets, int* work, int M, int E, int top, int groups, int keep, float scale,
                           int softmax, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  const int slots = top + (joint ? 1 : 0), all = E + (joint ? 1 : 0);
  if (bad_routing(M, E, top, groups, keep, slots)) return 10;
  if (joint && sg == nullptr) { set_error("moe_route: the joint expert needs its gate"); return 10; }
  if (ld < E) { set_error("moe_route: a logit per expert required"); return 10; }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const RouteParams p = {corr, weights, work + all, M, E, top, groups, keep, slots, scale, softmax ? SCORE_SOFTMAX : SCORE_SIGMOID};
  B2_DISPATCH_T(is_f32, moe_route_kernel<T><<<(M + MR_WARPS - 1) / MR_WARPS, MR_WARPS * 32, MR_WARPS * 2 * E * sizeof(float), st>>>(
      p, z, ld, sg, ld_sg););
  B2_CHECK_LAUNCH("moe_route");
  return launch_place(place, token, offsets, work, M, all, slots, st);
}

template <int FORM>
static int launch_skinny(const SkinnyParams& p, const RouteParams& r, cudaStream_t st) {
  const int nt = (p.N + 7) / 8;
  const dim3 wide((p.M + SK_ROWS - 1) / SK_ROWS, (p.N + 63) / 64), grid(wide.x);
  if constexpr (FORM == SK_TOKEN) {
    if (p.N <= 32) skinny_kernel<4, FORM><<<grid, SK_WARPS * 32, 0, st>>>(p, r);
    else skinny_kernel<8, FORM><<<wide, SK_WARPS * 32, 0, st>>>(p, r);
  } else {
#define B2_SKINNY(V) case V: skinny_kernel<V, FORM><<<grid, SK_WARPS * 32, 0, st>>>(p, r); break
    switch (nt) {
      B2_SKINNY(1); B2_SKINNY(2); B2_SKINNY(3); B2_SKINNY(4); B2_SKINNY(5); B2_SKINNY(6); B2_SKINNY(7); B2_SKINNY(8); B2_SKINNY(9);
      default: set_error("skinny: up to %d outputs", SK_MAX_TILES * 8); return 10;
    }
  }
#undef B2_SKINNY
  B2_CHECK_LAUNCH("skinny");
  return 0;
}

// z fp32 [M, N] (row stride ld_z) = h bf16 [M, K] w bf16 [N, K]^T for N up to 72
B2_EXPORT int b2_skinny(const void* h, long long ld_h, const void* w, long long ld_w, float* z, long long ld_z, int M, int N, int K,
                        void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (N < 1 || K < 8 || K % 8 || ld_h % 8 || ld_w % 8 || ld_z < N) { set_error("skinny: contraction and strides in multiples of 8 required"); return 10; }
  const SkinnyParams p = {static_cast<const moe_bf16*>(h), static_cast<const moe_bf16*>(w), z, ld_h, ld_w, ld_z, M, N, K, -1, nullptr, nullptr, nullptr, 0, 0, 0};
  return launch_skinny<SK_PLAIN>(p, RouteParams{}, static_cast<cudaStream_t>(stream));
}

// out bf16 [M, N] = gelu_tanh(h w^T) * table[ids, first ...]: for few rows; ids outside the vocabulary give zeros
B2_EXPORT int b2_token_gate(const void* h, long long ld_h, const void* w, long long ld_w, const void* table, long long ld_table,
                            const long long* ids, void* out, int M, int N, int K, int first, int vocab, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (N < 1 || K < 8 || K % 8 || ld_h % 8 || ld_w % 8 || first < 0 || first + N > ld_table) {
    set_error("token_gate: contraction and strides in multiples of 8 required");
    return 10;
  }
  const SkinnyParams p = {static_cast<const moe_bf16*>(h), static_cast<const moe_bf16*>(w), nullptr, ld_h, ld_w, 0, M, N, K, -1,
                          static_cast<const moe_bf16*>(table), ids, static_cast<moe_bf16*>(out), ld_table, first, vocab};
  return launch_skinny<SK_TOKEN>(p, RouteParams{}, static_cast<cudaStream_t>(stream));
}

// Router product and choice in one kernel, N = E router rows and what follows them in w (up to 72 rows); sg >= 0: row sg's product is
// the gate of the joint expert, or goes to sg_out fp32 [M].  The rest as b2_moe_route.
B2_EXPORT int b2_moe_router(const void* h, long long ld_h, const void* w, long long ld_w, int N, int K, int sg, float* sg_out,
                            int joint, const void* corr, float* weights, int* place, int* token, int* offsets, int* work, int M, int E, int top,
                            int groups, int keep, float scale, int softmax, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  const int slots = top + (joint ? 1 : 0), all = E + (joint ? 1 : 0);
  if (bad_routing(M, E, top, groups, keep, slots)) return 10;
  if (N < E || N > SK_MAX_TILES * 8 || K < 8 || K % 8 || ld_h % 8 || ld_w % 8 || sg >= N || (sg >= 0 && !joint && sg_out == nullptr) ||
      (joint && sg < 0)) {
    set_error("moe_router: up to %d outputs, contraction and strides in multiples of 8 required", SK_MAX_TILES * 8);
    return 10;
  }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const SkinnyParams p = {static_cast<const moe_bf16*>(h), static_cast<const moe_bf16*>(w), sg_out, ld_h, ld_w, 1, M, N, K, sg, nullptr, nullptr, nullptr, 0, 0, 0};
  const RouteParams r = {corr, weights, work + all, M, E, top, groups, keep, slots, scale, softmax ? SCORE_SOFTMAX : SCORE_SIGMOID};
  if (const int rc = launch_skinny<SK_ROUTE>(p, r, st)) return rc;
  return launch_place(place, token, offsets, work, M, all, slots, st);
}

// h: T [tokens, ld], w: T [E, 2, F, K], token: int32 [P] -> out T [P, F].  rows (bf16 [P, K], or null): room for the rows expert after
// expert, if they are to be laid out before the product.  clamped: the gated form with alpha and limit instead of silu.
B2_EXPORT int b2_moe_glu(const void* h, long long ld, const void* w, const int* token, const int* offsets, void* rows, void* out, int tokens,
                         int P, int E, int F, int K, int clamped, float alpha, float limit, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (P <= 0) return 0;
  if (E < 1 || E > MOE_MAX_EXPERTS || F < 8 || F % 8 || K < 8 || K % 8 || ld % 8 || ld < K || tokens < 1) {
    set_error("moe_glu: up to %d experts and sizes in multiples of 8 required", MOE_MAX_EXPERTS);
    return 10;
  }
  if (clamped && !(limit > 0.f)) { set_error("moe_glu: a positive limit required"); return 10; }
  const GluAct act = {clamped ? GLU_CLAMPED : GLU_SILU, alpha, limit};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (is_f32) {
    const int rows = moe_bound(P, E, MF_T);
    if (rows > 65535) { set_error("moe_glu: too many rows (%d)", P); return 10; }
    moe_gemm_f32_kernel<true><<<dim3((F + MF_T - 1) / MF_T, rows), 256, 0, st>>>(
        static_cast<const float*>(h), ld, static_cast<const float*>(w), token, offsets, static_cast<float*>(out), E, F, K, act);
    B2_CHECK_LAUNCH("moe_glu");
    return 0;
  }
  const uint64_t hd[2] = {static_cast<uint64_t>(K), static_cast<uint64_t>(tokens)}, hs[1] = {2ull * ld};
  const uint32_t hbox[2] = {MG_BK, 1};
  const MoeGemmParams p = {token, offsets, static_cast<moe_bf16*>(out), F, P, E, F, K, act};
  if (rows != nullptr) {
    const int blocks = (P + 7) / 8;
    moe_gather_kernel<<<blocks < 16 * num_sms() ? blocks : 16 * num_sms(), 256, 0, st>>>(static_cast<const moe_bf16*>(h), ld, token,
                                                                                        static_cast<moe_bf16*>(rows), tokens, P, K, status_ptr());
    B2_CHECK_LAUNCH("moe_gather");
    return launch_glu<ROWS_GLU>(tensor_map_2d_bf16(rows, P, K, K, MG_BM, MG_BK), w, p, moe_columns(P, E, F, 128, 32), moe_bound(P, E, MG_BM),
                                st);
  }
  return launch_glu<MOE_GLU>(tensor_map_nd_bf16(h, 2, hd, hs, hbox, 3), w, p, moe_columns(P, E, F, 128, 32), moe_bound(P, E, MG_BM), st);
}

// One feed-forward for all rows: h bf16 [M, ld], w bf16 [2, F, K] -> out bf16 [M, F] (row stride ld_out)
B2_EXPORT int b2_rows_glu(const void* h, long long ld, const void* w, void* out, long long ld_out, int M, int F, int K, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (F < 8 || F % 8 || K < 8 || K % 8 || ld % 8 || ld < K || ld_out % 8 || ld_out < F) {
    set_error("rows_glu: sizes and strides in multiples of 8 required");
    return 10;
  }
  const MoeGemmParams p = {nullptr, nullptr, static_cast<moe_bf16*>(out), ld_out, M, 1, F, K, {GLU_SILU, 0.f, 0.f}};
  return launch_glu<ROWS_GLU>(tensor_map_2d_bf16(h, M, K, ld, MG_BM, MG_BK), w, p, moe_columns(M, 1, F, 128, 32), (M + MG_BM - 1) / MG_BM,
                              static_cast<cudaStream_t>(stream));
}

// a: T [P, F], w: T [E, N, F] -> out T [P, N]
B2_EXPORT int b2_moe_down(const void* a, const void* w, const int* offsets, void* out, int P, int E, int N, int F, int is_f32,
                          void* stream) {
  b2::ensure_thread_context();
  if (P <= 0) return 0;
  if (E < 1 || E > MOE_MAX_EXPERTS || F < 8 || F % 8 || N < 8 || N % 8) {
    set_error("moe_down: up to %d experts and sizes in multiples of 8 required", MOE_MAX_EXPERTS);
    return 10;
  }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (is_f32) {
    const int rows = moe_bound(P, E, MF_T);
    if (rows > 65535) { set_error("moe_down: too many rows (%d)", P); return 10; }
    moe_gemm_f32_kernel<false><<<dim3((N + MF_T - 1) / MF_T, rows), 256, 0, st>>>(
        static_cast<const float*>(a), F, static_cast<const float*>(w), nullptr, offsets, static_cast<float*>(out), E, N, F, GluAct{});
    B2_CHECK_LAUNCH("moe_down");
    return 0;
  }
  const int cols = moe_columns(P, E, N, 256, 64);
  const uint64_t dims[3] = {static_cast<uint64_t>(F), static_cast<uint64_t>(N), static_cast<uint64_t>(E)},
                 strides[2] = {2ull * F, 2ull * N * F};
  const uint32_t box[3] = {MG_BK, static_cast<uint32_t>(cols), 1};
  const CUtensorMap *tb = tensor_map_nd_bf16(w, 3, dims, strides, box, 3), *ta = tensor_map_2d_bf16(a, P, F, F, MG_BM, MG_BK);
  if (!ta || !tb) return 2;
  const MoeGemmParams p = {nullptr, offsets, static_cast<moe_bf16*>(out), N, P, E, N, F, GluAct{}};
  const int bound = moe_bound(P, E, MG_BM);
  if (cols == 256) return launch_moe<256, MOE_DOWN>(ta, tb, p, bound, st);
  if (cols == 128) return launch_moe<128, MOE_DOWN>(ta, tb, p, bound, st);
  return launch_moe<64, MOE_DOWN>(ta, tb, p, bound, st);
}

B2_EXPORT int b2_moe_norm_add(float* x, const void* rows, const int* place, const float* weights, int top, int P, const float* shared,
                              const float* sg, int ld_sg, const void* w, void* h, int M, int ld, int n, float coef, float eps,
                              int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8 || n <= 0 || n > ld || ld > 32768 || top < 1 || top > MOE_MAX_TOP || (shared != nullptr && sg == nullptr)) {
    set_error("moe_norm_add: ld %% 8 == 0, 0 < n <= ld <= 32768 and up to %d rows a token required", MOE_MAX_TOP);
    return 10;
  }
  const MoeAddParams p = {x, rows, place, weights, shared, sg, w, h, top, P, ld_sg, ld, n, coef, eps, status_ptr()};
  const int pieces = ld / 8, V = pieces <= 256 ? 1 : pieces <= 512 ? 2 : 4;
  const int threads = ((pieces + V - 1) / V + 31) / 32 * 32;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  B2_DISPATCH_T(is_f32, {
    if (V == 1) moe_norm_add_kernel<T, 1, 256><<<M, threads, 0, st>>>(p);
    else if (V == 2) moe_norm_add_kernel<T, 2, 256><<<M, threads, 0, st>>>(p);
    else if (threads <= 256) moe_norm_add_kernel<T, 4, 256><<<M, threads, 0, st>>>(p);
    else moe_norm_add_kernel<T, 4, 1024><<<M, threads, 0, st>>>(p);
  });
  B2_CHECK_LAUNCH("moe_norm_add");
  return 0;
}
