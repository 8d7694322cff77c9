// Gated linear recurrence with one state per channel, behind a short causal convolution:
//
//   u = sum_j taps[K-1-j] (x + xb)[t-j] + cb            (zeros before the sequence's start)
//   r, i = sigmoid(z + zb)                              (z: block-diagonal products of u, made by head_linear)
//   log a = -8 r softplus(lam);   S <- a S + sqrt(1 - a^2) i u;   out = S gelu(y + yb)
//
// States are fp32 per sequence slot; start == 0 means that they are zero, whatever the slot holds.  Short portions are walked token by
// token.  Long ones are cut into chunks of 64 tokens: every chunk's own transfer (product of the decays, state from zero), the states
// at the chunks' starts, then the chunks once more from there.
#include "host.h"
#include "vec.cuh"

namespace b2 {

constexpr int GR_TILE = 16;          // rows of a convolution tile: at least taps - 1
constexpr int GR_THREADS = 128;
constexpr float GR_RATE = 8.f;

struct ConvParams {
  const void* x;         // T [M, ld]
  long long ld;
  const void* xb;        // T [C]
  const void* taps;      // T [C, K], last column: the current token
  const void* cb;        // T [C]
  float* state;          // [slots, C, K - 1] inputs, bias included
  void* u;               // T [M, C]
  const int* cu;
  const int* start;
  const int* slot;
  const int* tiles;      // [n, 4] = (sequence, first row, rows, offset in the portion)
  int C, K;
};

// Grid (tiles, channels / (8 * threads)), eight channels a thread.  Only the portion's first tile reads the state, so that tile also
// replaces it, after its own reads.
template <typename T>
__global__ void __launch_bounds__(GR_THREADS) causal_conv_kernel(const ConvParams p) {
  const int* tl = p.tiles + blockIdx.x * 4;
  const int s = tl[0], row0 = tl[1], rows = tl[2], off = tl[3], c = (blockIdx.y * GR_THREADS + threadIdx.x) * 8, K = p.K;
  const int slot = s < 0 ? -1 : p.slot[s];
  if (slot < 0 || rows <= 0 || c >= p.C) return;
  const bool fresh = p.start[s] == 0;
  const T* x = static_cast<const T*>(p.x) + c;
  const T* taps = static_cast<const T*>(p.taps) + static_cast<size_t>(c) * K;
  float* st = p.state + (static_cast<size_t>(slot) * p.C + c) * (K - 1);
  float xb[8], cb[8];
  vload8(static_cast<const T*>(p.xb) + c, xb);
  vload8(static_cast<const T*>(p.cb) + c, cb);
  auto input = [&](int at, float (&f)[8]) {          // input at index `at` of the portion
    if (at >= 0) {
      vload8(x + (static_cast<size_t>(row0) + at - off) * p.ld, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] += xb[e];
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = fresh ? 0.f : st[e * (K - 1) + K - 1 + at];
    }
  };
  for (int t = 0; t < rows; ++t) {
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = cb[e];
    for (int j = 0; j < K; ++j) {
      float f[8];
      input(off + t - j, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = fmaf(to_f(taps[e * K + K - 1 - j]), f[e], acc[e]);
    }
    vstore8(static_cast<T*>(p.u) + (static_cast<size_t>(row0) + t) * p.C + c, acc);
  }
  if (off != 0 || K < 2) return;
  const int count = p.cu[s + 1] - p.cu[s];
  for (int j = 0; j < K - 1; ++j) {                  // in this order an old input is read before its place is written
    float f[8];
    input(count - (K - 1) + j, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) st[e * (K - 1) + j] = f[e];
  }
}

struct RecParams {
  const void* u;         // T [M, ld_u]
  const float* z;        // [M, ld_z]: per block the recurrence gate's columns, then the input gate's
  const void* zb;        // T, in the same order
  const void* lam;       // T [C]
  const void* y;         // T [M, ld_y]
  const void* yb;        // T [C]
  void* out;             // T [M, ld_out]
  float* state;          // [slots, C]
  float* ws;             // [chunks, 2, C]: transfer (product, end state), then [.., 0, ..] the state at the chunk's start
  const int* cu;
  const int* start;
  const int* slot;
  const int* chunks;     // [n, 4]
  const int* first;      // [nlong + 1]
  long long ld_u, ld_z, ld_y, ld_out;
  int C, block, seq0;
};

// 1 - e^x for x <= 0, accurate near zero
__device__ __forceinline__ float one_minus_exp(float x, float ex) {
  if (x > -0.125f) {
    float t = fmaf(x, 1.f / 720.f, 1.f / 120.f);
    t = fmaf(x, t, 1.f / 24.f);
    t = fmaf(x, t, 1.f / 6.f);
    t = fmaf(x, t, 0.5f);
    t = fmaf(x, t, 1.f);
    return -x * t;
  }
  return 1.f - ex;
}

// decay and increment of one channel and token; sp = GR_RATE * softplus(lam)
template <typename T>
__device__ __forceinline__ float2 rec_step(float zr, float zi, float u, float sp) {
  const float x = -sp * sigmoid_t<T>(zr);
  float a, m;
  if (sizeof(T) == 2) {
    a = fast_exp2(1.4426950408889634f * x);
    m = one_minus_exp(2.f * x, a * a);
  } else {
    a = expf(x);
    m = -expm1f(2.f * x);
  }
  return make_float2(a, sqrtf(m) * sigmoid_t<T>(zi) * u);
}

// A channel's place: its gates' columns and constants.
template <typename T>
struct RecChannel {
  int c, zc;
  float sp, br, bi, yb;
  __device__ __forceinline__ RecChannel(const RecParams& p, int ch) : c(ch) {
    zc = ch / p.block * 2 * p.block + ch % p.block;
    sp = GR_RATE * softplus_f(to_f(static_cast<const T*>(p.lam)[ch]));
    br = to_f(static_cast<const T*>(p.zb)[zc]);
    bi = to_f(static_cast<const T*>(p.zb)[zc + p.block]);
    yb = to_f(static_cast<const T*>(p.yb)[ch]);
  }
  __device__ __forceinline__ float2 step(const RecParams& p, size_t row) const {
    const float* z = p.z + row * p.ld_z + zc;
    return rec_step<T>(z[0] + br, z[p.block] + bi, to_f(static_cast<const T*>(p.u)[row * p.ld_u + c]), sp);
  }
};

template <typename T>
__global__ void __launch_bounds__(GR_THREADS) rec_transfer_kernel(const RecParams p) {
  const int* ch = p.chunks + blockIdx.x * 4;
  const int c = blockIdx.y * GR_THREADS + threadIdx.x;
  if (c >= p.C || p.slot[ch[0]] < 0) return;
  const RecChannel<T> k(p, c);
  float A = 1.f, S = 0.f;
#pragma unroll 4
  for (int t = 0; t < ch[2]; ++t) {
    const float2 g = k.step(p, static_cast<size_t>(ch[1]) + t);
    A *= g.x;
    S = fmaf(g.x, S, g.y);
  }
  float* w = p.ws + static_cast<size_t>(blockIdx.x) * 2 * p.C + c;
  w[0] = A;
  w[p.C] = S;
}

// Grid (channels, long sequences)
__global__ void __launch_bounds__(GR_THREADS) rec_carry_kernel(const RecParams p) {
  const int c = blockIdx.x * GR_THREADS + threadIdx.x, s = p.seq0 + blockIdx.y;
  const int slot = p.slot[s];
  if (c >= p.C || slot < 0) return;
  float* st = p.state + static_cast<size_t>(slot) * p.C + c;
  float S = p.start[s] == 0 ? 0.f : *st;
  const int c0 = p.first[blockIdx.y], c1 = p.first[blockIdx.y + 1];
  constexpr int U = 8;
  for (int i = c0; i < c1; i += U) {
    float A[U], B[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const float* w = p.ws + static_cast<size_t>(min(i + u, c1 - 1)) * 2 * p.C + c;
      A[u] = w[0];
      B[u] = w[p.C];
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (i + u >= c1) break;
      p.ws[static_cast<size_t>(i + u) * 2 * p.C + c] = S;
      S = fmaf(A[u], S, B[u]);
    }
  }
  *st = S;
}

// CHUNKS: grid (chunks, channels), from the states rec_carry left; else grid (sequences, channels), from the slots and back to them.
template <typename T, bool CHUNKS>
__global__ void __launch_bounds__(GR_THREADS) rec_out_kernel(const RecParams p) {
  const int c = blockIdx.y * GR_THREADS + threadIdx.x;
  const int s = CHUNKS ? p.chunks[blockIdx.x * 4] : p.seq0 + static_cast<int>(blockIdx.x);
  const int slot = p.slot[s];
  if (c >= p.C || slot < 0) return;
  const size_t row0 = CHUNKS ? p.chunks[blockIdx.x * 4 + 1] : p.cu[s];
  const int rows = CHUNKS ? p.chunks[blockIdx.x * 4 + 2] : p.cu[s + 1] - p.cu[s];
  float* st = p.state + static_cast<size_t>(slot) * p.C + c;
  float S = CHUNKS ? p.ws[static_cast<size_t>(blockIdx.x) * 2 * p.C + c] : p.start[s] == 0 ? 0.f : *st;
  const RecChannel<T> k(p, c);
#pragma unroll 4
  for (int t = 0; t < rows; ++t) {
    const size_t row = row0 + t;
    const float2 g = k.step(p, row);
    const float y = gelu_tanh_t<T>(to_f(static_cast<const T*>(p.y)[row * p.ld_y + c]) + k.yb);
    S = fmaf(g.x, S, g.y);
    static_cast<T*>(p.out)[row * p.ld_out + c] = from_f<T>(S * y);
  }
  if (!CHUNKS) *st = S;
}

}  // namespace b2

using namespace b2;

B2_EXPORT int b2_causal_conv(const void* x, long long ld, const void* xb, const void* taps, const void* cb, float* state, void* u,
                             const int* cu, const int* start, const int* slot, const int* tiles, int ntiles, int C, int K,
                             int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (ntiles <= 0) return 0;
  if (C < 8 || C % 8 || ld % 8 || K < 1 || K - 1 > GR_TILE) {
    set_error("causal_conv: channels in multiples of 8 and 1 to %d taps required", GR_TILE + 1);
    return 10;
  }
  const ConvParams p = {x, ld, xb, taps, cb, state, u, cu, start, slot, tiles, C, K};
  const dim3 grid(ntiles, (C / 8 + GR_THREADS - 1) / GR_THREADS);
  B2_DISPATCH_T(is_f32, causal_conv_kernel<T><<<grid, GR_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(p););
  B2_CHECK_LAUNCH("causal_conv");
  return 0;
}

// Sequences seq0 .. seq0 + nseq - 1; nchunks > 0: they are long, chunks / first describe them and ws is fp32 [nchunks, 2, C].
B2_EXPORT int b2_linear_recurrence(const void* u, long long ld_u, const float* z, long long ld_z, const void* zb, const void* lam,
                                   const void* y, long long ld_y, const void* yb, void* out, long long ld_out, float* state, float* ws,
                                   const int* cu, const int* start, const int* slot, const int* chunks, const int* first, int nchunks,
                                   int seq0, int nseq, int C, int block, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (nseq <= 0) return 0;
  if (C < 1 || block < 1 || C % block || nseq > 65535 || (nchunks > 0 && (ws == nullptr || chunks == nullptr || first == nullptr))) {
    set_error("linear_recurrence: channels in equal blocks required");
    return 10;
  }
  const RecParams p = {u, z, zb, lam, y, yb, out, state, ws, cu, start, slot, chunks, first, ld_u, ld_z, ld_y, ld_out, C, block, seq0};
  const int cy = (C + GR_THREADS - 1) / GR_THREADS;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (nchunks > 0) {
    B2_DISPATCH_T(is_f32, rec_transfer_kernel<T><<<dim3(nchunks, cy), GR_THREADS, 0, st>>>(p););
    B2_CHECK_LAUNCH("rec_transfer");
    rec_carry_kernel<<<dim3(cy, nseq), GR_THREADS, 0, st>>>(p);
    B2_CHECK_LAUNCH("rec_carry");
    B2_DISPATCH_T(is_f32, (rec_out_kernel<T, true><<<dim3(nchunks, cy), GR_THREADS, 0, st>>>(p)););
  } else {
    B2_DISPATCH_T(is_f32, (rec_out_kernel<T, false><<<dim3(nseq, cy), GR_THREADS, 0, st>>>(p)););
  }
  B2_CHECK_LAUNCH("linear_recurrence");
  return 0;
}
