// Latent attention: what is cached of a token is one row for all heads, a normed latent c and a rotated key part
//
//   [ c (kv_rank, padded to Cp) | rotated part (padded) ]      pages [blocks, 16, Rp], Rp = Cp + padded rotated size
//
// from which a head's key is [W_uk c | rotated part] and its value W_uv c.  Two ways to attend, equal but for rounding:
//   expanded   keys and values of all heads are made from the rows (a GEMM) and attended like ordinary ones: long portions, where
//              a row serves many queries (latent_gather brings the pages into token order for that GEMM)
//   absorbed   q_h^T W_uk c = (W_uk^T q_h)^T c, so the query moves into the latent space, every head attends over the same rows,
//              and W_uv is applied to the result: decoding and short portions (between two products per head, head_linear); in
//              bf16 by the kernel of attention_decode.cu, in 32-bit and for sizes beyond it by latent_rows here
// And the stage before either: norm of the latent (and of the one queries are made from, where they have one), rotary positions of the
// queries' and the key's rotated part, page store.  Queries made from a latent are turned later: by the product that moves them into
// the latent space, or in place for the expanded way (latent_turn).  A window limits how far back a query sees; a gate per head
// scales its output.
#include "host.h"
#include "mma_split.cuh"
#include "vec.cuh"

namespace b2 {

constexpr int LA_PAGE = 16;
constexpr float LA_LOG2E = 1.4426950408889634f;
typedef __nv_bfloat16 la_bf16;

__device__ __forceinline__ void la_copy16(void* dst, const void* src, bool in) {
  const int n = in ? 16 : 0;   // zero-filled otherwise
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void la_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void la_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// ---- input stage -----------------------------------------------------------------------------------------------------------
// The rotated part of a row's queries: channels dim .. dim + rot - 1 of every head, pairs (2 i, 2 i + 1).
constexpr int LS_THREADS = 128;
template <typename T>
__device__ __forceinline__ void turn_heads(T* qr, const float* cr, const float* sr, int H, int dim, int dqp, int rot) {
  const int tid = threadIdx.x, half = rot / 2;
  if (dim % 8 == 0 && rot % 8 == 0) {        // four pairs at a time
    const int per = rot / 8;
    for (int i = tid; i < H * per; i += LS_THREADS) {
      const int h = i / per, f = i % per * 4;
      T* at = qr + static_cast<size_t>(h) * dqp + dim + 2 * f;
      float t[8];
      vload8(at, t);
      const float4 co = *reinterpret_cast<const float4*>(cr + f), si = *reinterpret_cast<const float4*>(sr + f);
      const float c4[4] = {co.x, co.y, co.z, co.w}, s4[4] = {si.x, si.y, si.z, si.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float u = t[2 * e], v = t[2 * e + 1];
        t[2 * e] = u * c4[e] - v * s4[e];
        t[2 * e + 1] = v * c4[e] + u * s4[e];
      }
      vstore8(at, t);
    }
  } else {
    for (int i = tid; i < H * half; i += LS_THREADS) {
      const int h = i / half, f = i % half;
      T* at = qr + static_cast<size_t>(h) * dqp + dim + 2 * f;
      const float u = to_f(at[0]), v = to_f(at[1]), co = cr[f], si = sr[f];
      at[0] = from_f<T>(u * co - v * si);
      at[1] = from_f<T>(v * co + u * si);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(LS_THREADS) latent_turn_kernel(T* __restrict__ q, long long ld, const float* __restrict__ cs,
                                                                 const float* __restrict__ sn, int H, int dim, int dqp, int rot) {
  const size_t row = blockIdx.x;
  turn_heads(q + row * ld, cs + row * (rot / 2), sn + row * (rot / 2), H, dim, dqp, rot);
}

struct LatentStoreParams {
  void* q;               // T [M, ld] H * dqp columns, turned in place, or null
  void* cq;              // T [M, ld] Qp columns, normed in place (weight wq, q_rank real channels), or null
  const void* c;         // T [M, ld] Cp columns
  const void* kr;        // T [M, ld] Rp - Cp columns
  void* pages;
  const void *w, *wq;
  const int *tables, *row_seq, *pos, *slot;
  const float *cs, *sn;
  long long ld;
  int max_blocks, H, dim, dqp, rank, Cp, Rp, rot, q_rank, Qp;
  float eps;
};

// One row per CTA.
template <typename T>
__global__ void __launch_bounds__(LS_THREADS) latent_store_kernel(const LatentStoreParams p) {
  __shared__ float red[2][LS_THREADS / 32];
  const size_t row = blockIdx.x;
  const int s = p.row_seq ? p.row_seq[row] : static_cast<int>(row), tid = threadIdx.x, half = p.rot / 2;
  const float* cr = p.cs + row * half;
  const float* sr = p.sn + row * half;
  if (p.q) turn_heads(static_cast<T*>(p.q) + row * p.ld, cr, sr, p.H, p.dim, p.dqp, p.rot);
  const T* crow = static_cast<const T*>(p.c) + row * p.ld;
  T* qrow = static_cast<T*>(p.cq) + row * p.ld;
  auto sum_squares = [&](const T* v, int n) {
    float ss = 0.f;
    for (int a = tid * 8; a < n; a += LS_THREADS * 8) {
      float t[8];
      vload8(v + a, t);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(t[e], t[e], ss);
    }
    return warp_sum(ss);
  };
  auto scaled = [&](const T* v, const T* w, T* dst, int n, float r) {
    for (int a = tid * 8; a < n; a += LS_THREADS * 8) {
      float t[8], g[8];
      vload8(v + a, t);
      vload8(w + a, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) t[e] *= r * g[e];
      vstore8(dst + a, t);
    }
  };
  const float ss = sum_squares(crow, p.Cp), sq = p.cq ? sum_squares(qrow, p.Qp) : 0.f;
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = ss;
    red[1][tid >> 5] = sq;
  }
  __syncthreads();
  if (p.cq)
    scaled(qrow, static_cast<const T*>(p.wq), qrow, p.Qp, 1.f / sqrtf((red[1][0] + red[1][1] + red[1][2] + red[1][3]) / p.q_rank + p.eps));
  if (p.slot != nullptr && p.slot[s] < 0) return;
  const int pos = p.pos[row];
  T* dst = static_cast<T*>(p.pages) + (static_cast<size_t>(p.tables[static_cast<size_t>(s) * p.max_blocks + pos / LA_PAGE]) * LA_PAGE +
                                       pos % LA_PAGE) * p.Rp;
  scaled(crow, static_cast<const T*>(p.w), dst, p.Cp, 1.f / sqrtf((red[0][0] + red[0][1] + red[0][2] + red[0][3]) / p.rank + p.eps));
  const T* krow = static_cast<const T*>(p.kr) + row * p.ld;
  for (int f = LS_THREADS - 1 - tid; f < (p.Rp - p.Cp) / 2; f += LS_THREADS) {
    float u = to_f(krow[2 * f]), v = to_f(krow[2 * f + 1]);
    if (f < half) {
      const float x = u * cr[f] - v * sr[f];
      v = v * cr[f] + u * sr[f];
      u = x;
    }
    dst[p.Cp + 2 * f] = from_f<T>(u);
    dst[p.Cp + 2 * f + 1] = from_f<T>(v);
  }
}

// out page i <- page ids[i], `bytes` a page
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint8_t* __restrict__ pages, const int* __restrict__ ids,
                                                            uint8_t* __restrict__ out, int bytes) {
  const uint8_t* src = pages + static_cast<size_t>(ids[blockIdx.x]) * bytes;
  uint8_t* dst = out + static_cast<size_t>(blockIdx.x) * bytes;
  for (int i = threadIdx.x * 16; i < bytes; i += 128 * 16)
    *reinterpret_cast<uint4*>(dst + i) = *reinterpret_cast<const uint4*>(src + i);
}

// ---- one small product per head ----------------------------------------------------------------------------------------------
// out[m, h, :] = W_h x[m, h, :] with W_h [N, K] (KN: W_h stored [K, N]); x rows of stride ld_x with heads xs apart, out likewise.  On
// the 32-bit result: columns turn_at .. turn_at + 2 half - 1 turned in pairs by the row's angles (cs given), the head's columns
// times sigmoid(gate[m, h]) (gate given).
struct HeadLinearParams {
  const void* x;
  const void* w;
  void* out;
  long long ld_x, ld_out;
  int M, H, N, K, xs, os;
  const float *cs, *sn;  // [M, half]
  const void* gate;      // type of x, [M, ld_gate]
  long long ld_gate;
  int turn_at, half;
};

template <bool KN>
__global__ void __launch_bounds__(256) head_linear_any_kernel(const HeadLinearParams p) {
  const int n = blockIdx.x * 256 + threadIdx.x, h = blockIdx.y;
  const float* w = static_cast<const float*>(p.w) + static_cast<size_t>(h) * p.N * p.K;
  if (n >= p.N) return;
  for (int m = blockIdx.z; m < p.M; m += gridDim.z) {
    const float* x = static_cast<const float*>(p.x) + m * p.ld_x + static_cast<size_t>(h) * p.xs;
    auto dot = [&](int col) {
      float s = 0.f;
      for (int k = 0; k < p.K; ++k) s = fmaf(x[k], KN ? w[static_cast<size_t>(k) * p.N + col] : w[static_cast<size_t>(col) * p.K + k], s);
      return s;
    };
    float s = dot(n);
    const int f = n - p.turn_at;
    if (p.cs != nullptr && f >= 0 && f < 2 * p.half) {
      const float other = dot(p.turn_at + (f ^ 1)), co = p.cs[static_cast<size_t>(m) * p.half + f / 2], si = p.sn[static_cast<size_t>(m) * p.half + f / 2];
      s = f & 1 ? s * co + other * si : s * co - other * si;
    }
    if (p.gate != nullptr) s *= sigmoid_f(static_cast<const float*>(p.gate)[m * p.ld_gate + h]);
    static_cast<float*>(p.out)[m * p.ld_out + static_cast<size_t>(h) * p.os + n] = s;
  }
}

// bf16: a 64 x 64 output tile of one head per CTA, four warps of 16 rows, K in pieces of 64 through two stages.
constexpr int HL_T = 64, HL_LD = HL_T + 8;
// O: type of the result
template <bool KN, typename O>
__global__ void __launch_bounds__(128) head_linear_kernel(const HeadLinearParams p) {
  __shared__ __align__(16) la_bf16 sA[2][HL_T][HL_LD], sB[2][HL_T][HL_LD];
  const int n0 = blockIdx.x * HL_T, h = blockIdx.y, m0 = blockIdx.z * HL_T;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const la_bf16* x = static_cast<const la_bf16*>(p.x) + static_cast<size_t>(h) * p.xs;
  const la_bf16* w = static_cast<const la_bf16*>(p.w) + static_cast<size_t>(h) * p.N * p.K;
  auto issue = [&](int st, int k0) {
    for (int i = tid; i < HL_T * (HL_T / 8); i += 128) {
      const int r = i / 8, c = i % 8 * 8;
      const bool ia = m0 + r < p.M && k0 + c < p.K;
      la_copy16(&sA[st][r][c], x + (ia ? (m0 + r) * p.ld_x + k0 + c : 0), ia);
      const int n = KN ? n0 + c : n0 + r, k = KN ? k0 + r : k0 + c;
      const bool ib = n < p.N && k < p.K;
      la_copy16(&sB[st][r][c], w + (ib ? (KN ? static_cast<size_t>(k) * p.N + n : static_cast<size_t>(n) * p.K + k) : 0), ib);
    }
    la_commit();
  };
  float acc[HL_T / 8][4] = {};
  issue(0, 0);
  int st = 0;
  for (int k0 = 0; k0 < p.K; k0 += HL_T, st ^= 1) {
    if (k0 + HL_T < p.K) {
      issue(st ^ 1, k0 + HL_T);
      la_wait<1>();
    } else {
      la_wait<0>();
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < HL_T / 16; ++ks) {
      uint32_t a[4];
      ldsm_a_mk(&sA[st][warp * 16][ks * 16], HL_LD, lane, a);
#pragma unroll
      for (int n = 0; n < HL_T; n += 16) {
        uint32_t b[4];
        if (KN) ldsm_b_kn(&sB[st][ks * 16][n], HL_LD, lane, b);
        else ldsm_b_nk(&sB[st][n][ks * 16], HL_LD, lane, b);
        mma_n16(acc[n / 8], acc[n / 8 + 1], a, b);
      }
    }
    __syncthreads();
  }
  O* out = static_cast<O*>(p.out) + static_cast<size_t>(h) * p.os;
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    const int m = m0 + warp * 16 + (lane >> 2) + 8 * hh;
    if (m >= p.M) continue;
    const float g = p.gate ? sigmoid_fast(to_f(static_cast<const la_bf16*>(p.gate)[m * p.ld_gate + h])) : 1.f;
#pragma unroll
    for (int n = 0; n < HL_T / 8; ++n) {
      const int c = n0 + n * 8 + (lane & 3) * 2;
      if (c >= p.N) continue;
      float u = acc[n][2 * hh] * g, v = acc[n][2 * hh + 1] * g;
      const int f = (c - p.turn_at) / 2;
      if (p.cs != nullptr && c >= p.turn_at && f < p.half) {
        const float co = p.cs[static_cast<size_t>(m) * p.half + f], si = p.sn[static_cast<size_t>(m) * p.half + f], t = u * co - v * si;
        v = v * co + u * si;
        u = t;
      }
      if (sizeof(O) == 4) *reinterpret_cast<float2*>(out + m * p.ld_out + c) = make_float2(u, v);
      else *reinterpret_cast<uint32_t*>(out + m * p.ld_out + c) = pack_bf16x2(u, v);
    }
  }
}

// ---- absorbed attention ------------------------------------------------------------------------------------------------------
struct LatentRowsParams {
  const void* q;         // T [M, H * Rp]
  const void* pages;     // T [blocks, 16, Rp]
  const int* tables;
  const int* row_seq;    // [M] or null: row r is sequence r
  const int* pos;
  const int* slot;       // slot < 0: padding row (output zero)
  const void* sink;      // T [H] or null
  void* out;             // T [M, H * Cp]
  float* part_o;         // [M, H, nsplit, Cp]
  float* part_ml;        // [M, H, nsplit, 2]
  int max_blocks, H, Rp, Cp, partition, nsplit;
  int window;            // > 0: keys pos - window + 1 .. pos; partitions count from the first visible key
  float scale;
};

template <typename T>
__device__ __forceinline__ float la_sink(const LatentRowsParams& p, int head, float M2, float L) {
  // factor on the weighted sum of values: 1 / (L + sink), M2 being the maximum in the base-2 domain
  if (p.sink == nullptr) return L > 0.f ? 1.f / L : 0.f;
  const float s2 = to_f(static_cast<const T*>(p.sink)[head]) * LA_LOG2E, m = fmaxf(M2, s2);
  const float w = M2 == -INFINITY ? 0.f : exp2f(M2 - m);
  return w / (L * w + exp2f(s2 - m));
}

// Any sizes, any type: one CTA per (row, head, split); a key per warp at a time, its channels over the lanes.
constexpr int LR_ANY_WARPS = 4;
template <typename T, int E>
__global__ void __launch_bounds__(LR_ANY_WARPS * 32) latent_rows_any_kernel(const LatentRowsParams p) {
  extern __shared__ __align__(16) float la_any[];     // q [32 E], then accumulators [warps][32 E]
  __shared__ float sM[LR_ANY_WARPS], sL[LR_ANY_WARPS];
  const size_t row = blockIdx.x;
  const int head = blockIdx.y, split = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int s = p.row_seq ? p.row_seq[row] : static_cast<int>(row);
  const bool live = p.slot == nullptr || p.slot[s] >= 0;
  const int seen = p.window > 0 ? max(0, p.pos[row] - p.window + 1) : 0;
  const int t_begin = seen + split * p.partition, t_end = live ? min(p.pos[row] + 1, t_begin + p.partition) : t_begin;
  const int* table = p.tables + static_cast<size_t>(s) * p.max_blocks;
  const T* q = static_cast<const T*>(p.q) + (row * p.H + head) * p.Rp;
  float* sQ = la_any;
  float* sAcc = la_any + 32 * E;
  for (int c = threadIdx.x; c < 32 * E; c += LR_ANY_WARPS * 32) sQ[c] = c < p.Rp ? to_f(q[c]) * (p.scale * LA_LOG2E) : 0.f;
  __syncthreads();
  float acc[E], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int e = 0; e < E; ++e) acc[e] = 0.f;
  for (int t = t_begin + warp; t < t_end; t += LR_ANY_WARPS) {
    const T* k = static_cast<const T*>(p.pages) + (static_cast<size_t>(table[t / LA_PAGE]) * LA_PAGE + t % LA_PAGE) * p.Rp;
    float v[E], d = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int c = lane + 32 * e;
      v[e] = c < p.Rp ? to_f(k[c]) : 0.f;
      d = fmaf(v[e], sQ[c], d);
    }
    d = warp_sum(d);
    const float mn = fmaxf(m, d), a = exp2f(m - mn), w = exp2f(d - mn);
    m = mn;
    l = l * a + w;
#pragma unroll
    for (int e = 0; e < E; ++e) acc[e] = acc[e] * a + w * v[e];
  }
#pragma unroll
  for (int e = 0; e < E; ++e) sAcc[warp * 32 * E + lane + 32 * e] = acc[e];
  if (lane == 0) {
    sM[warp] = m;
    sL[warp] = l;
  }
  __syncthreads();
  float M = -INFINITY, L = 0.f;
  for (int w = 0; w < LR_ANY_WARPS; ++w) M = fmaxf(M, sM[w]);
  for (int w = 0; w < LR_ANY_WARPS; ++w) L += sM[w] == -INFINITY ? 0.f : sL[w] * exp2f(sM[w] - M);
  const size_t at = (row * p.H + head) * p.nsplit + split;
  const float f = p.nsplit == 1 ? la_sink<T>(p, head, M, L) : 1.f;
  for (int c = threadIdx.x; c < p.Cp; c += LR_ANY_WARPS * 32) {
    float o = 0.f;
    for (int w = 0; w < LR_ANY_WARPS; ++w) o += sM[w] == -INFINITY ? 0.f : sAcc[w * 32 * E + c] * exp2f(sM[w] - M);
    if (p.nsplit == 1) static_cast<T*>(p.out)[(row * p.H + head) * p.Cp + c] = from_f<T>(o * f);
    else p.part_o[at * p.Cp + c] = o;
  }
  if (p.nsplit > 1 && threadIdx.x == 0) {
    p.part_ml[at * 2] = M;
    p.part_ml[at * 2 + 1] = L;
  }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentRowsParams p) {
  const size_t row = blockIdx.x;
  const int head = blockIdx.y;
  const size_t at = (row * p.H + head) * p.nsplit;
  float M = -INFINITY, L = 0.f;
  for (int i = 0; i < p.nsplit; ++i) M = fmaxf(M, p.part_ml[(at + i) * 2]);
  for (int i = 0; i < p.nsplit; ++i) {
    const float mi = p.part_ml[(at + i) * 2];
    L += mi == -INFINITY ? 0.f : p.part_ml[(at + i) * 2 + 1] * exp2f(mi - M);
  }
  const float f = la_sink<T>(p, head, M, L);
  for (int c = threadIdx.x * 8; c < p.Cp; c += 128 * 8) {
    float o[8] = {};
    for (int i = 0; i < p.nsplit; ++i) {
      const float mi = p.part_ml[(at + i) * 2];
      if (mi == -INFINITY) continue;
      const float w = exp2f(mi - M);
      float t[8];
      vload8(p.part_o + (at + i) * p.Cp + c, t);
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] = fmaf(t[e], w, o[e]);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] *= f;
    vstore8(static_cast<T*>(p.out) + (row * p.H + head) * p.Cp + c, o);
  }
}

}  // namespace b2

using namespace b2;

// q null: the queries are made later, from cq (Qp columns of which q_rank are real), which is normed here
B2_EXPORT int b2_latent_store(void* q, void* cq, const void* c, const void* kr, long long ld, void* pages, const void* w, const void* wq,
                              const int* tables, const int* row_seq, const int* pos, const int* slot, const float* cs, const float* sn,
                              int M, int max_blocks, int H, int dim, int dqp, int rank, int Cp, int Rp, int rot, int q_rank, int Qp,
                              float eps, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (rot < 2 || rot % 2 || Cp % 8 || Rp % 8 || rank < 1 || rank > Cp || Rp - Cp < rot || ld % 8 || max_blocks < 1 ||
      (q != nullptr && (H < 1 || dim < 1 || dim + rot > dqp || dqp % 8)) ||
      (cq != nullptr && (wq == nullptr || q_rank < 1 || q_rank > Qp || Qp % 8))) {
    set_error("latent_store: padded sizes in multiples of 8 and an even rotated size required");
    return 10;
  }
  const LatentStoreParams p = {q, cq, c, kr, pages, w, wq, tables, row_seq, pos, slot, cs, sn, ld, max_blocks, H, dim, dqp, rank, Cp, Rp, rot,
                               q_rank, Qp, eps};
  B2_DISPATCH_T(is_f32, latent_store_kernel<T><<<M, LS_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(p););
  B2_CHECK_LAUNCH("latent_store");
  return 0;
}

// q [M, ld]: the rotated part of every head, in place
B2_EXPORT int b2_latent_turn(void* q, long long ld, const float* cs, const float* sn, int M, int H, int dim, int dqp, int rot, int is_f32,
                             void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (H < 1 || dim < 1 || rot < 2 || rot % 2 || dim + rot > dqp || dqp % 8 || ld % 8) {
    set_error("latent_turn: padded sizes in multiples of 8 and an even rotated size required");
    return 10;
  }
  B2_DISPATCH_T(is_f32, latent_turn_kernel<T><<<M, LS_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(static_cast<T*>(q), ld, cs, sn, H, dim,
                                                                                                      dqp, rot););
  B2_CHECK_LAUNCH("latent_turn");
  return 0;
}

// ids: int32 [n] page of the pool for every page of out; page_bytes a multiple of 16
B2_EXPORT int b2_latent_gather(const void* pages, const int* ids, void* out, int n, int page_bytes, void* stream) {
  b2::ensure_thread_context();
  if (n <= 0) return 0;
  if (page_bytes < 16 || page_bytes % 16) { set_error("latent_gather: pages of a multiple of 16 bytes required"); return 10; }
  latent_gather_kernel<<<n, 128, 0, static_cast<cudaStream_t>(stream)>>>(static_cast<const uint8_t*>(pages), ids,
                                                                         static_cast<uint8_t*>(out), page_bytes);
  B2_CHECK_LAUNCH("latent_gather");
  return 0;
}

// out_f32: a 32-bit result of bf16 operands; cs, sn, gate: see HeadLinearParams
B2_EXPORT int b2_head_linear(const void* x, const void* w, void* out, long long ld_x, long long ld_out, int M, int H, int N, int K,
                             int xs, int os, int kn, const float* cs, const float* sn, int turn_at, int half, const void* gate,
                             long long ld_gate, int is_f32, int out_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (H < 1 || H > 65535 || N < 8 || K < 8 || N % 8 || K % 8 || xs % 8 || os % 8 || ld_x % 8 || ld_out % 8) {
    set_error("head_linear: sizes and strides in multiples of 8 required");
    return 10;
  }
  if (cs != nullptr && (sn == nullptr || half < 1 || turn_at < 0 || turn_at % 2 || turn_at + 2 * half > N)) {
    set_error("head_linear: turned columns outside the result");
    return 10;
  }
  HeadLinearParams p = {x, w, out, ld_x, ld_out, M, H, N, K, xs, os, cs, sn, gate, ld_gate, turn_at, half};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (is_f32) {
    const dim3 grid((N + 255) / 256, H, M < 65535 ? M : 65535);
    if (kn) head_linear_any_kernel<true><<<grid, 256, 0, st>>>(p);
    else head_linear_any_kernel<false><<<grid, 256, 0, st>>>(p);
  } else {
    const dim3 grid((N + HL_T - 1) / HL_T, H, (M + HL_T - 1) / HL_T);
    if (grid.z > 65535) { set_error("head_linear: too many rows (%d)", M); return 10; }
    if (out_f32) {
      if (kn) head_linear_kernel<true, float><<<grid, 128, 0, st>>>(p);
      else head_linear_kernel<false, float><<<grid, 128, 0, st>>>(p);
    } else {
      if (kn) head_linear_kernel<true, la_bf16><<<grid, 128, 0, st>>>(p);
      else head_linear_kernel<false, la_bf16><<<grid, 128, 0, st>>>(p);
    }
  }
  B2_CHECK_LAUNCH("head_linear");
  return 0;
}

// partition: keys per split; nsplit * partition must cover every row's visible keys.
B2_EXPORT int b2_latent_rows(const void* q, const void* pages, const int* tables, const int* row_seq, const int* pos,
                             const int* slot, const void* sink, void* out, float* part_o, float* part_ml, int M, int max_blocks,
                             int H, int Rp, int Cp, int partition, int nsplit, int window, float scale, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (H < 1 || H > 65535 || Rp % 8 || Cp % 8 || Cp < 8 || Rp < Cp || Rp > 1280 || partition < 1 || nsplit < 1 || nsplit > 65535 ||
      max_blocks < 1 || (nsplit > 1 && (part_o == nullptr || part_ml == nullptr))) {
    set_error("latent_rows: rows up to 1280 channels in multiples of 8 required");
    return 10;
  }
  LatentRowsParams p = {q, pages, tables, row_seq, pos, slot, sink, out, part_o, part_ml, max_blocks, H, Rp, Cp, partition, nsplit,
                        window, scale};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 grid(M, H, nsplit);
  B2_DISPATCH_T(is_f32, {
    if (Rp <= 256) {
      latent_rows_any_kernel<T, 8><<<grid, LR_ANY_WARPS * 32, 5 * 256 * 4, st>>>(p);
    } else {
      latent_rows_any_kernel<T, 40><<<grid, LR_ANY_WARPS * 32, 5 * 1280 * 4, st>>>(p);
    }
  });
  B2_CHECK_LAUNCH("latent_rows");
  if (nsplit > 1) {
    B2_DISPATCH_T(is_f32, latent_merge_kernel<T><<<dim3(M, H), 128, 0, st>>>(p););
    B2_CHECK_LAUNCH("latent_merge");
  }
  return 0;
}
