// Kernels around a 32-bit residual stream: embedding into it (of the token alone, or of the token and of the pair it forms with the one
// before, normed), RMS norm or layer norm out of it, the half-sum of two normed branches added to it (with the next norm in the same
// pass), one normed branch added to it (plain, or gated, layer-normed and scaled per channel with the next layer norm in the same
// pass), gated activations over column slices or with a table of per-token vectors, rotary tables for a batch's positions, and the
// 32-bit matrix product used when a model runs without any reduced-precision mode.
//
// Rows of the residual and of every activation are padded to a multiple of eight columns; `n` is the real width.  The
// padding columns are zero (their norm weights are zero), so vector accesses never need a tail.
#include "host.h"
#include "vec.cuh"

namespace b2 {

constexpr int RES_THREADS = 256;
constexpr int RES_VEC = 4;   // 8-column pieces a thread keeps in registers (rows up to 8192 columns); longer rows are re-read

__device__ __forceinline__ float res_block_sum(float v, float* scratch) {
  v = warp_sum(v);
  __syncthreads();   // the previous use of scratch has been read
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  const int lane = threadIdx.x & 31;
  return warp_sum(lane < static_cast<int>(blockDim.x >> 5) ? scratch[lane] : 0.f);
}

template <typename T>
__global__ void __launch_bounds__(RES_THREADS) embed_f32_kernel(const long long* __restrict__ ids, const T* __restrict__ table,
                                                                float* __restrict__ x, T* __restrict__ h, int ld, int vocab,
                                                                float scale) {
  const long long id = ids[blockIdx.x];
  const bool ok = id >= 0 && id < vocab;   // padding rows of a graph batch carry any id; nothing outside the table is read
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
    float f[8] = {};
    if (ok) vload8(table + static_cast<size_t>(id) * ld + c, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= scale;
    vstore8(x + static_cast<size_t>(blockIdx.x) * ld + c, f);
    if (h) vstore8(h + static_cast<size_t>(blockIdx.x) * ld + c, f);
  }
}

template <typename T>
__global__ void __launch_bounds__(RES_THREADS) rmsnorm_f32_kernel(const float* __restrict__ x, const T* __restrict__ w,
                                                                  T* __restrict__ h, const long long* __restrict__ rows, int ld,
                                                                  int n, float eps, float scale) {
  __shared__ float scratch[32];
  const size_t src = rows ? static_cast<size_t>(rows[blockIdx.x]) : blockIdx.x;
  const float* xr = x + src * ld;
  T* hr = h + static_cast<size_t>(blockIdx.x) * ld;
  float v[RES_VEC][8], ss = 0.f;
  int i = 0;
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8, ++i) {
    float t[8];
    vload8(xr + c, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(t[e], t[e], ss);
#pragma unroll
    for (int k = 0; k < RES_VEC; ++k)
      if (k == i)
#pragma unroll
        for (int e = 0; e < 8; ++e) v[k][e] = t[e];
  }
  const float r = scale / sqrtf(res_block_sum(ss, scratch) / n + eps);
  i = 0;
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8, ++i) {
    float t[8], wv[8];
    if (i >= RES_VEC) vload8(xr + c, t);
#pragma unroll
    for (int k = 0; k < RES_VEC; ++k)
      if (k == i)
#pragma unroll
        for (int e = 0; e < 8; ++e) t[e] = v[k][e];
    vload8(w + c, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) t[e] *= r * wv[e];
    vstore8(hr + c, t);
  }
}

// x <- rms(alpha x + f y + b) w, and the same rounded to T in h (optional).  y: fp32 [M, ld]; b (optional): T [ld]; f is 1, or
// the root of a norm over the reader's input that was left to this kernel: 1 / sqrt(sum_j ss[row, j] / nss + eps).
template <typename T>
__global__ void __launch_bounds__(RES_THREADS) post_norm_kernel(float* __restrict__ x, const float* __restrict__ y,
                                                                const T* __restrict__ w, const T* __restrict__ b,
                                                                const float* __restrict__ ss, int parts, int nss,
                                                                T* __restrict__ h, int ld, int n, float alpha, float eps) {
  __shared__ float scratch[32];
  const size_t base = static_cast<size_t>(blockIdx.x) * ld;
  float f = 1.f;
  if (ss) {
    float t = 0.f;
    for (int j = 0; j < parts; ++j) t += ss[static_cast<size_t>(blockIdx.x) * parts + j];
    f = 1.f / sqrtf(t / nss + eps);
  }
  auto piece = [&](int c, float (&s)[8]) {
    float t[8];
    vload8(x + base + c, s);
    vload8(y + base + c, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) s[e] = fmaf(alpha, s[e], f * t[e]);
    if (b) {
      vload8(b + c, t);
#pragma unroll
      for (int e = 0; e < 8; ++e) s[e] += t[e];
    }
  };
  float v[RES_VEC][8], sum = 0.f;
  int i = 0;
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8, ++i) {
    float t[8];
    piece(c, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) sum = fmaf(t[e], t[e], sum);
#pragma unroll
    for (int k = 0; k < RES_VEC; ++k)
      if (k == i)
#pragma unroll
        for (int e = 0; e < 8; ++e) v[k][e] = t[e];
  }
  const float r = 1.f / sqrtf(res_block_sum(sum, scratch) / n + eps);
  i = 0;
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8, ++i) {
    float t[8], wv[8];
    if (i >= RES_VEC) piece(c, t);
#pragma unroll
    for (int k = 0; k < RES_VEC; ++k)
      if (k == i)
#pragma unroll
        for (int e = 0; e < 8; ++e) t[e] = v[k][e];
    vload8(w + c, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) t[e] *= r * wv[e];
    vstore8(x + base + c, t);
    if (h) vstore8(h + base + c, t);
  }
}

// x += coef * (rms(a) wa + rms(b) wb); h = rms(x) w_next when w_next is given.  a, b: fp32 [M, ld].
template <typename T>
__global__ void __launch_bounds__(RES_THREADS) merge_norm_add_kernel(float* __restrict__ x, const float* __restrict__ a,
                                                                     const float* __restrict__ b, const T* __restrict__ wa,
                                                                     const T* __restrict__ wb, const T* __restrict__ w_next,
                                                                     T* __restrict__ h, int ld, int n, float coef, float eps) {
  __shared__ float scratch[32];
  const size_t base = static_cast<size_t>(blockIdx.x) * ld;
  float sa = 0.f, sb = 0.f;
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
    float t[8], u[8];
    vload8(a + base + c, t);
    vload8(b + base + c, u);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      sa = fmaf(t[e], t[e], sa);
      sb = fmaf(u[e], u[e], sb);
    }
  }
  const float ra = coef / sqrtf(res_block_sum(sa, scratch) / n + eps);
  const float rb = coef / sqrtf(res_block_sum(sb, scratch) / n + eps);
  float ss = 0.f;
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
    float t[8], u[8], f[8], va[8], vb[8];
    vload8(a + base + c, t);
    vload8(b + base + c, u);
    vload8(wa + c, va);
    vload8(wb + c, vb);
    vload8(x + base + c, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      f[e] += t[e] * ra * va[e] + u[e] * rb * vb[e];
      ss = fmaf(f[e], f[e], ss);
    }
    vstore8(x + base + c, f);
  }
  if (w_next == nullptr) return;
  const float r = 1.f / sqrtf(res_block_sum(ss, scratch) / n + eps);
  for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {   // re-reads what this thread just wrote
    float f[8], wv[8];
    vload8(x + base + c, f);
    vload8(w_next + c, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= r * wv[e];
    vstore8(h + base + c, f);
  }
}

// x += coef * rms(f y) * w, and the new x rounded to T in h (optional).  y: fp32 [M, ld].  A row's pieces (V per thread) stay in
// registers; both rows are requested before the first is used.
template <typename T, int V, int MAXT>
__global__ void __launch_bounds__(MAXT) norm_add_kernel(float* __restrict__ x, const float* __restrict__ y, const T* __restrict__ w,
                                                        T* __restrict__ h, int ld, int n, float coef, float eps, float f) {
  __shared__ float scratch[32];
  const size_t base = static_cast<size_t>(blockIdx.x) * ld;
  float a[V][8], b[V][8], ss = 0.f;
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
#pragma unroll
    for (int e = 0; e < 8; ++e) a[k][e] = b[k][e] = 0.f;
    if (c < ld) {
      vload8(y + base + c, a[k]);
      vload8(x + base + c, b[k]);
    }
  }
#pragma unroll
  for (int k = 0; k < V; ++k)
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      a[k][e] *= f;
      ss = fmaf(a[k][e], a[k][e], ss);
    }
  const float r = coef / sqrtf(res_block_sum(ss, scratch) / n + eps);
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c >= ld) break;
    float wv[8];
    vload8(w + c, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) b[k][e] = fmaf(a[k][e] * r, wv[e], b[k][e]);
    vstore8(x + base + c, b[k]);
    if (h) vstore8(h + base + c, b[k]);
  }
}

// ---- layer norms ---------------------------------------------------------------------------------------------------------------
// A row lies in the registers of a block, V pieces of eight channels a thread, zero past its n channels.  The mean is taken off
// before anything is squared.
__device__ __forceinline__ float row_sum(float v, float* scratch) {      // scratch: 32 floats that nothing else uses
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  const int lane = threadIdx.x & 31;
  return warp_sum(lane < static_cast<int>(blockDim.x >> 5) ? scratch[lane] : 0.f);
}
__device__ __forceinline__ int row_piece(int k) { return (threadIdx.x + k * blockDim.x) * 8; }

// a <- (a - mean) / sqrt(variance + eps)
template <int V>
__device__ __forceinline__ void row_standardise(float (&a)[V][8], int n, float eps, float (*scratch)[32]) {
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < V; ++k)
#pragma unroll
    for (int e = 0; e < 8; ++e) s += a[k][e];
  const float mean = row_sum(s, scratch[0]) / n;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < V; ++k)
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      a[k][e] = row_piece(k) + e < n ? a[k][e] - mean : 0.f;
      ss = fmaf(a[k][e], a[k][e], ss);
    }
  const float r = 1.f / sqrtf(row_sum(ss, scratch[1]) / n + eps);
#pragma unroll
  for (int k = 0; k < V; ++k)
#pragma unroll
    for (int e = 0; e < 8; ++e) a[k][e] *= r;
}

// a <- a * w + b, the weights' padding being zero
template <typename T, int V>
__device__ __forceinline__ void row_affine(float (&a)[V][8], const T* w, const T* b, int ld) {
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = row_piece(k);
    if (c >= ld) break;
    float wv[8], bv[8];
    vload8(w + c, wv);
    vload8(b + c, bv);
#pragma unroll
    for (int e = 0; e < 8; ++e) a[k][e] = fmaf(a[k][e], wv[e], bv[e]);
  }
}
template <typename T, int V>
__device__ __forceinline__ void row_store(const float (&a)[V][8], T* dst, int ld) {
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = row_piece(k);
    if (c >= ld) break;
    vstore8(dst + c, a[k]);
  }
}

// h = layer norm of x[rows]
template <typename T, int V, int MAXT>
__global__ void __launch_bounds__(MAXT) layernorm_f32_kernel(const float* __restrict__ x, const T* __restrict__ w, const T* __restrict__ b,
                                                             T* __restrict__ h, const long long* __restrict__ rows, int ld, int n,
                                                             float eps) {
  __shared__ float scratch[2][32];
  const float* xr = x + (rows ? static_cast<size_t>(rows[blockIdx.x]) : blockIdx.x) * ld;
  float a[V][8];
#pragma unroll
  for (int k = 0; k < V; ++k) {
#pragma unroll
    for (int e = 0; e < 8; ++e) a[k][e] = 0.f;
    if (row_piece(k) < ld) vload8(xr + row_piece(k), a[k]);
  }
  row_standardise(a, n, eps, scratch);
  row_affine(a, w, b, ld);
  row_store(a, h + static_cast<size_t>(blockIdx.x) * ld, ld);
}

// x = layer norm of table[id] + pairs[(before * mul_prev + id * mul_cur) mod buckets], `before` the sequence's token before this one; the
// first token of a sequence takes row `buckets` of pairs.  h = layer norm of x with the reader's weights.  Between steps the last
// token of a sequence waits in its slot: the block of the portion's first row reads it and puts the portion's last token there.
struct EmbedPairsParams {
  const long long* ids;
  const void *table, *pairs;
  int* last;             // [slots]
  const int *cu, *row_seq, *pos, *slot;
  const void *w, *b, *next_w, *next_b;
  float* x;
  void* h;
  long long mul_prev, mul_cur, buckets;
  int ld, n, vocab;
  float eps;
};
template <typename T, int V, int MAXT>
__global__ void __launch_bounds__(MAXT) embed_pairs_kernel(const EmbedPairsParams p) {
  __shared__ float scratch[4][32];
  const int row = blockIdx.x, s = p.row_seq[row], first = p.cu[s], slot = p.slot[s];
  const long long id = p.ids[row];
  const bool ok = id >= 0 && id < p.vocab;      // padding rows of a graph batch carry any id; nothing outside the tables is read
  long long pair = p.buckets;
  if (p.pos[row] > 0) {
    const long long before = row > first ? p.ids[row - 1] : slot >= 0 ? p.last[slot] : 0;
    pair = (before * p.mul_prev + id * p.mul_cur) % p.buckets;
    if (pair < 0) pair += p.buckets;
  }
  const T* tr = static_cast<const T*>(p.table) + static_cast<size_t>(ok ? id : 0) * p.ld;
  const T* pr = static_cast<const T*>(p.pairs) + static_cast<size_t>(pair) * p.ld;
  float a[V][8];
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = row_piece(k);
#pragma unroll
    for (int e = 0; e < 8; ++e) a[k][e] = 0.f;
    if (c >= p.ld || !ok) continue;
    float t[8];
    vload8(tr + c, a[k]);
    vload8(pr + c, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) a[k][e] += t[e];
  }
  row_standardise(a, p.n, p.eps, scratch);      // its barriers: every thread has read `last`
  if (row == first && slot >= 0 && threadIdx.x == 0) p.last[slot] = static_cast<int>(p.ids[p.cu[s + 1] - 1]);
  row_affine(a, static_cast<const T*>(p.w), static_cast<const T*>(p.b), p.ld);
  row_store(a, p.x + static_cast<size_t>(row) * p.ld, p.ld);
  if (p.h == nullptr) return;
  row_standardise(a, p.n, p.eps, scratch + 2);
  row_affine(a, static_cast<const T*>(p.next_w), static_cast<const T*>(p.next_b), p.ld);
  row_store(a, static_cast<T*>(p.h) + static_cast<size_t>(row) * p.ld, p.ld);
}

// x += s * layer norm(y * sigmoid(gate + gate_b)), h = layer norm of the new x with the reader's weights.  y: fp32 rows, or (ROWS) the
// weighted sum of a token's expert rows.  Gate and s are optional.
constexpr int BA_MAX_TOP = 32;
struct BranchParams {
  float* x;              // [M, ld]
  const float* y;        // [M, ld]
  const void* rows;      // ROWS: T [P, ld]
  const int* place;      // [M, top]
  const float* weights;  // [M, top]
  const void* gate;      // G [M, ld_gate] or null
  const void *gate_b, *w, *b, *s, *next_w, *next_b;     // T [ld]; gate_b with gate, s or null, next_* with h
  void* h;               // T [M, ld] or null
  long long ld_gate;
  int top, P, ld, n;
  float eps;
  int* status;
};
template <typename T, typename G, int V, int MAXT, bool ROWS>
__global__ void __launch_bounds__(MAXT) branch_add_kernel(const BranchParams p) {
  __shared__ float scratch[4][32], sw[BA_MAX_TOP];
  __shared__ int sr[BA_MAX_TOP];
  const size_t base = static_cast<size_t>(blockIdx.x) * p.ld;
  if (ROWS) {
    if (static_cast<int>(threadIdx.x) < p.top) {
      sw[threadIdx.x] = p.weights[static_cast<size_t>(blockIdx.x) * p.top + threadIdx.x];
      int r = p.place[static_cast<size_t>(blockIdx.x) * p.top + threadIdx.x];
      if (r < 0 || r >= p.P) {                  // an index that came from memory: recorded, and the access left out
        atomicCAS(p.status, 0, ERR_BAD_ARGUMENT);
        r = 0;
      }
      sr[threadIdx.x] = r;
    }
    __syncthreads();
  }
  const T* rows = static_cast<const T*>(p.rows);
  float a[V][8], x[V][8];
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = row_piece(k);
#pragma unroll
    for (int e = 0; e < 8; ++e) a[k][e] = x[k][e] = 0.f;
    if (c >= p.ld) continue;
    vload8(p.x + base + c, x[k]);
    float g[8] = {}, gb[8] = {};
    if (p.gate) {
      vload8(static_cast<const G*>(p.gate) + blockIdx.x * p.ld_gate + c, g);
      vload8(static_cast<const T*>(p.gate_b) + c, gb);
    }
    if (ROWS) {
      for (int j = 0; j < p.top; j += 4) {
        Packed8<T> t[4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (j + i < p.top) t[i].load(rows + static_cast<size_t>(sr[j + i]) * p.ld + c);
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (j + i < p.top) {
            float f[8];
            t[i].get(f);
#pragma unroll
            for (int e = 0; e < 8; ++e) a[k][e] = fmaf(sw[j + i], f[e], a[k][e]);
          }
      }
    } else {
      vload8(p.y + base + c, a[k]);
    }
    if (p.gate)
#pragma unroll
      for (int e = 0; e < 8; ++e) a[k][e] *= sigmoid_t<T>(g[e] + gb[e]);
  }
  row_standardise(a, p.n, p.eps, scratch);
  row_affine(a, static_cast<const T*>(p.w), static_cast<const T*>(p.b), p.ld);
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int c = row_piece(k);
    if (c >= p.ld) break;
    float f[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
    if (p.s) vload8(static_cast<const T*>(p.s) + c, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[k][e] = fmaf(a[k][e], f[e], x[k][e]);
  }
  row_store(x, p.x + base, p.ld);
  if (p.h == nullptr) return;
  row_standardise(x, p.n, p.eps, scratch + 2);
  row_affine(x, static_cast<const T*>(p.next_w), static_cast<const T*>(p.next_b), p.ld);
  row_store(x, static_cast<T*>(p.h) + base, p.ld);
}

// A block for a row of ld channels: pieces a thread and threads; FN<V, MAXT>
#define B2_ROW_LAUNCH(ld, ...)                                                          \
  do {                                                                                  \
    const int pieces_ = (ld) / 8, v_ = pieces_ <= 256 ? 1 : pieces_ <= 512 ? 2 : 4;     \
    const int threads = ((pieces_ + v_ - 1) / v_ + 31) / 32 * 32;                       \
    if (v_ == 1) { constexpr int V = 1, MAXT = 256; __VA_ARGS__; }                      \
    else if (v_ == 2) { constexpr int V = 2, MAXT = 256; __VA_ARGS__; }                 \
    else if (threads <= 256) { constexpr int V = 4, MAXT = 256; __VA_ARGS__; }          \
    else { constexpr int V = 4, MAXT = 1024; __VA_ARGS__; }                             \
  } while (0)

// out = gelu_tanh(gate) * table[id, first ...]: ids outside the vocabulary (padding rows) give zeros
template <typename T>
__global__ void __launch_bounds__(RES_THREADS) gelu_token_kernel(const T* __restrict__ gate, const T* __restrict__ table,
                                                                 const long long* __restrict__ ids, T* __restrict__ out, int n,
                                                                 int ld_gate, long long ld_table, int first, int vocab, long long total) {
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long row = i / (n / 8);
    const int c = static_cast<int>(i - row * (n / 8)) * 8;
    const long long id = ids[row];
    float g[8], t[8] = {};
    vload8(gate + row * ld_gate + c, g);
    if (id >= 0 && id < vocab) vload8(table + id * ld_table + first + c, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] = gelu_tanh_t<T>(g[e]) * t[e];
    vstore8(out + row * n + c, g);
  }
}

// out = silu(gate) * up over column slices (row strides ld_in / ld_out)
template <typename T>
__global__ void __launch_bounds__(RES_THREADS) glu_kernel(const T* __restrict__ gate, const T* __restrict__ up,
                                                          T* __restrict__ out, int ld_in, int ld_out, int nvec, long long total) {
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long row = i / nvec;
    const int c = static_cast<int>(i - row * nvec) * 8;
    float g[8], u[8];
    vload8(gate + row * ld_in + c, g);
    vload8(up + row * ld_in + c, u);
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] = silu_t<T>(g[e]) * u[e];
    vstore8(out + row * ld_out + c, g);
  }
}

// cos / sin of position * freq, the angle reduced in double precision: turns[i] = freq_i / (2 pi).
__global__ void __launch_bounds__(RES_THREADS) rope_rows_kernel(const int* __restrict__ pos, const double* __restrict__ turns,
                                                                float* __restrict__ cs, float* __restrict__ sn, int half,
                                                                int total) {
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < total; i += gridDim.x * blockDim.x) {
    const double t = static_cast<double>(pos[i / half]) * turns[i % half];
    float s, c;
    sincospif(2.f * static_cast<float>(t - rint(t)), &s, &c);
    cs[i] = c;
    sn[i] = s;
  }
}

// C[M,N] (+)= A[M,K] B[N,K]^T in plain fp32 FMA (64 x 64 tile, 4 x 4 per thread).
constexpr int SG_T = 64, SG_K = 16;
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ B,
                                                       float* __restrict__ C, int M, int N, int K, int lda, int ldb, int ldc,
                                                       int accumulate, int act, int act_cols) {
  __shared__ float sA[SG_K][SG_T + 4], sB[SG_K][SG_T + 4];
  const int m0 = blockIdx.y * SG_T, n0 = blockIdx.x * SG_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += SG_K) {
    for (int i = threadIdx.x; i < SG_T * SG_K; i += 256) {
      const int r = i / SG_K, k = i % SG_K;
      const bool in = k0 + k < K;
      sA[k][r] = in && m0 + r < M ? A[static_cast<size_t>(m0 + r) * lda + k0 + k] : 0.f;
      sB[k][r] = in && n0 + r < N ? B[static_cast<size_t>(n0 + r) * ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sA[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sB[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float* c = C + static_cast<size_t>(m) * ldc + n;
      float r = accumulate ? *c + acc[i][j] : acc[i][j];
      if (act != 0 && n < act_cols) r = act == GEMM_ACT_SILU ? silu_f(r) : fmaxf(r, 0.f) * fmaxf(r, 0.f);
      *c = r;
    }
  }
}

}  // namespace b2

using namespace b2;

// h (optional): the same rows in the table's type.
B2_EXPORT int b2_embed_f32(const long long* ids, const void* table, float* x, void* h, int M, int ld, int vocab, float scale,
                           int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8) { set_error("embed_f32: row width must be a multiple of 8"); return 10; }
  B2_DISPATCH_T(is_f32, embed_f32_kernel<T><<<M, RES_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(
      ids, static_cast<const T*>(table), x, static_cast<T*>(h), ld, vocab, scale););
  B2_CHECK_LAUNCH("embed_f32");
  return 0;
}

B2_EXPORT int b2_rmsnorm_f32(const float* x, const void* w, void* h, const long long* rows, int M, int ld, int n, float eps,
                             float scale, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8 || n <= 0 || n > ld) { set_error("rmsnorm_f32: ld %% 8 == 0 and 0 < n <= ld required"); return 10; }
  B2_DISPATCH_T(is_f32, rmsnorm_f32_kernel<T><<<M, RES_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(
      x, static_cast<const T*>(w), static_cast<T*>(h), rows, ld, n, eps, scale););
  B2_CHECK_LAUNCH("rmsnorm_f32");
  return 0;
}

B2_EXPORT int b2_post_norm(float* x, const float* y, const void* w, const void* b, const float* ss, int parts, int nss, void* h,
                           int M, int ld, int n, float alpha, float eps, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8 || n <= 0 || n > ld || (ss != nullptr && (parts < 1 || nss < 1))) {
    set_error("post_norm: ld %% 8 == 0 and 0 < n <= ld required");
    return 10;
  }
  int threads = (ld / 8 + 31) / 32 * 32;
  if (threads > RES_THREADS) threads = RES_THREADS;
  B2_DISPATCH_T(is_f32, post_norm_kernel<T><<<M, threads, 0, static_cast<cudaStream_t>(stream)>>>(
      x, y, static_cast<const T*>(w), static_cast<const T*>(b), ss, parts, nss, static_cast<T*>(h), ld, n, alpha, eps););
  B2_CHECK_LAUNCH("post_norm");
  return 0;
}

B2_EXPORT int b2_norm_add(float* x, const float* y, const void* w, void* h, int M, int ld, int n, float coef, float eps, float y_scale,
                          int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8 || n <= 0 || n > ld || ld > 32768) { set_error("norm_add: ld %% 8 == 0, 0 < n <= ld <= 32768 required"); return 10; }
  const int pieces = ld / 8, V = pieces <= 256 ? 1 : pieces <= 512 ? 2 : 4;
  const int threads = ((pieces + V - 1) / V + 31) / 32 * 32;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  B2_DISPATCH_T(is_f32, {
    const T* wt = static_cast<const T*>(w);
    T* ht = static_cast<T*>(h);
    if (V == 1) norm_add_kernel<T, 1, 256><<<M, threads, 0, st>>>(x, y, wt, ht, ld, n, coef, eps, y_scale);
    else if (V == 2) norm_add_kernel<T, 2, 256><<<M, threads, 0, st>>>(x, y, wt, ht, ld, n, coef, eps, y_scale);
    else if (threads <= 256) norm_add_kernel<T, 4, 256><<<M, threads, 0, st>>>(x, y, wt, ht, ld, n, coef, eps, y_scale);
    else norm_add_kernel<T, 4, 1024><<<M, threads, 0, st>>>(x, y, wt, ht, ld, n, coef, eps, y_scale);
  });
  B2_CHECK_LAUNCH("norm_add");
  return 0;
}

// gate [M, n] (row stride ld_gate), table rows of stride ld_table; n, first and the strides multiples of 8
B2_EXPORT int b2_gelu_token(const void* gate, const void* table, const long long* ids, void* out, int M, int n, int ld_gate,
                            long long ld_table, int first, int vocab, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (n < 8 || n % 8 || ld_gate % 8 || ld_table % 8 || first % 8 || first < 0 || first + n > ld_table) {
    set_error("gelu_token: columns and strides must be multiples of 8");
    return 10;
  }
  const long long total = static_cast<long long>(M) * (n / 8);
  long long blocks = (total + RES_THREADS - 1) / RES_THREADS;
  const long long cap = static_cast<long long>(num_sms()) * 16;
  if (blocks > cap) blocks = cap;
  B2_DISPATCH_T(is_f32, gelu_token_kernel<T><<<static_cast<int>(blocks), RES_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const T*>(gate), static_cast<const T*>(table), ids, static_cast<T*>(out), n, ld_gate, ld_table, first, vocab, total););
  B2_CHECK_LAUNCH("gelu_token");
  return 0;
}

B2_EXPORT int b2_merge_norm_add(float* x, const float* a, const float* b, const void* wa, const void* wb, const void* w_next,
                                void* h, int M, int ld, int n, float coef, float eps, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8 || n <= 0 || n > ld) { set_error("merge_norm_add: ld %% 8 == 0 and 0 < n <= ld required"); return 10; }
  B2_DISPATCH_T(is_f32, merge_norm_add_kernel<T><<<M, RES_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(
      x, a, b, static_cast<const T*>(wa), static_cast<const T*>(wb), static_cast<const T*>(w_next), static_cast<T*>(h), ld, n,
      coef, eps););
  B2_CHECK_LAUNCH("merge_norm_add");
  return 0;
}

B2_EXPORT int b2_glu(const void* gate, const void* up, void* out, int M, int cols, int ld_in, int ld_out, int is_f32,
                     void* stream) {
  b2::ensure_thread_context();
  if (M <= 0 || cols <= 0) return 0;
  if (cols % 8 || ld_in % 8 || ld_out % 8) { set_error("glu: columns and strides must be multiples of 8"); return 10; }
  const long long total = static_cast<long long>(M) * (cols / 8);
  long long blocks = (total + RES_THREADS - 1) / RES_THREADS;
  const long long cap = static_cast<long long>(num_sms()) * 16;
  if (blocks > cap) blocks = cap;
  B2_DISPATCH_T(is_f32, glu_kernel<T><<<static_cast<int>(blocks), RES_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const T*>(gate), static_cast<const T*>(up), static_cast<T*>(out), ld_in, ld_out, cols / 8, total););
  B2_CHECK_LAUNCH("glu");
  return 0;
}

B2_EXPORT int b2_rope_rows(const int* pos, const double* turns, float* cs, float* sn, int M, int half, void* stream) {
  b2::ensure_thread_context();
  const long long total = static_cast<long long>(M) * half;
  if (total <= 0) return 0;
  if (total > 0x7fffffffll) { set_error("rope_rows: too many rows"); return 10; }
  long long blocks = (total + RES_THREADS - 1) / RES_THREADS;
  const long long cap = static_cast<long long>(num_sms()) * 8;
  if (blocks > cap) blocks = cap;
  rope_rows_kernel<<<static_cast<int>(blocks), RES_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(
      pos, turns, cs, sn, half, static_cast<int>(total));
  B2_CHECK_LAUNCH("rope_rows");
  return 0;
}

B2_EXPORT int b2_gemm_f32(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc,
                          int accumulate, int act, int act_cols, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  const dim3 grid((N + SG_T - 1) / SG_T, (M + SG_T - 1) / SG_T);
  if (grid.y > 65535) { set_error("gemm_f32: too many rows (%d)", M); return 10; }
  gemm_f32_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(A, B, C, M, N, K, lda, ldb, ldc, accumulate, act,
                                                                     act_cols);
  B2_CHECK_LAUNCH("gemm_f32");
  return 0;
}

B2_EXPORT int b2_layernorm_f32(const float* x, const void* w, const void* b, void* h, const long long* rows, int M, int ld, int n, float eps,
                               int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8 || n <= 0 || n > ld || ld > 32768) { set_error("layernorm_f32: ld %% 8 == 0, 0 < n <= ld <= 32768 required"); return 10; }
  B2_DISPATCH_T(is_f32, B2_ROW_LAUNCH(ld, (layernorm_f32_kernel<T, V, MAXT><<<M, threads, 0, static_cast<cudaStream_t>(stream)>>>(
      x, static_cast<const T*>(w), static_cast<const T*>(b), static_cast<T*>(h), rows, ld, n, eps))););
  B2_CHECK_LAUNCH("layernorm_f32");
  return 0;
}

// table T [vocab, ld], pairs T [buckets + 1, ld], last int32 [slots] (slot < 0: a padding row), h and next_* together or not at all
B2_EXPORT int b2_embed_pairs(const long long* ids, const void* table, const void* pairs, int* last, const int* cu, const int* row_seq,
                             const int* pos, const int* slot, const void* w, const void* b, const void* next_w, const void* next_b, float* x,
                             void* h, int M, int ld, int n, int vocab, long long buckets, long long mul_prev, long long mul_cur, float eps,
                             int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8 || n <= 0 || n > ld || ld > 32768 || vocab < 1 || buckets < 1 || (h != nullptr && (next_w == nullptr || next_b == nullptr))) {
    set_error("embed_pairs: ld %% 8 == 0, 0 < n <= ld <= 32768 and a bucket required");
    return 10;
  }
  const EmbedPairsParams p = {ids, table, pairs, last, cu, row_seq, pos, slot, w, b, next_w, next_b, x, h, mul_prev, mul_cur, buckets, ld, n, vocab, eps};
  B2_DISPATCH_T(is_f32, B2_ROW_LAUNCH(ld, (embed_pairs_kernel<T, V, MAXT><<<M, threads, 0, static_cast<cudaStream_t>(stream)>>>(p))););
  B2_CHECK_LAUNCH("embed_pairs");
  return 0;
}

// rows given: the weighted sum of top rows a token (P rows in all) in place of y.  gate_f32: a 32-bit gate beside bf16 weights.
B2_EXPORT int b2_branch_add(float* x, const float* y, const void* rows, const int* place, const float* weights, int top, int P, const void* gate,
                            long long ld_gate, int gate_f32, const void* gate_b, const void* w, const void* b, const void* s, const void* next_w,
                            const void* next_b, void* h, int M, int ld, int n, float eps, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (ld % 8 || n <= 0 || n > ld || ld > 32768 || (rows == nullptr) == (y == nullptr) ||
      (rows != nullptr && (top < 1 || top > BA_MAX_TOP || place == nullptr || weights == nullptr)) ||
      (gate != nullptr && (gate_b == nullptr || ld_gate % 8)) || (h != nullptr && (next_w == nullptr || next_b == nullptr))) {
    set_error("branch_add: ld %% 8 == 0, 0 < n <= ld <= 32768 and up to %d rows a token required", BA_MAX_TOP);
    return 10;
  }
  int* status = status_ptr();
  if (!status) return 3;
  const BranchParams p = {x, y, rows, place, weights, gate, gate_b, w, b, s, next_w, next_b, h, ld_gate, top, P, ld, n, eps, status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  B2_DISPATCH_T(is_f32, B2_ROW_LAUNCH(ld, {
    if (rows != nullptr) {
      if (gate_f32) branch_add_kernel<T, float, V, MAXT, true><<<M, threads, 0, st>>>(p);
      else branch_add_kernel<T, T, V, MAXT, true><<<M, threads, 0, st>>>(p);
    } else {
      if (gate_f32) branch_add_kernel<T, float, V, MAXT, false><<<M, threads, 0, st>>>(p);
      else branch_add_kernel<T, T, V, MAXT, false><<<M, threads, 0, st>>>(p);
    }
  }););
  B2_CHECK_LAUNCH("branch_add");
  return 0;
}
