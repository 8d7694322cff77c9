// Gated linear recurrence with one state per channel, behind a short causal convolution:
//
//   u = sum_j taps[K-1-j] (x + xb)[t-j] + cb            (zeros before the sequence's start)
//   r, i = sigmoid(z + zb)                              (z: block-diagonal products of u, made by head_linear)
//   log a = -8 r softplus(lam);   S <- a S + sqrt(1 - a^2) i u;   out = S gelu(y + yb)
//
// States are fp32 per sequence slot; start == 0 means that they are zero, whatever the slot holds.  Short portions are walked token by
// token.  Long ones are cut into runs of 32 tokens: every run's own transfer (product of the decays, state from zero), the states
// at the runs' starts, then the runs once more from there.  In bf16 the gates of both passes are tcgen05 products inside the pass
// (rec_gates_kernel): the accumulators have a channel per TMEM lane and a token per column, so that a thread finds the gates of its
// channel's tokens in its own lane and the recurrence never leaves registers; gates are made twice instead of stored.
#include <type_traits>

#include "host.h"
#include "vec.cuh"

namespace b2 {

constexpr int GR_TILE = 16;          // rows of a convolution tile: at least taps - 1
constexpr int GR_THREADS = 128;
constexpr float GR_RATE = 8.f;

struct ConvParams {
  const void* x;         // T [M, ld]
  long long ld;
  const void* xb;        // T [C] or null
  const void* taps;      // T [C, K], last column: the current token
  const void* cb;        // T [C] or null
  float* state;          // [slots, C, K - 1] inputs, bias included
  void* u;               // T [M, C]
  const int* cu;
  const int* start;
  const int* slot;
  const int* tiles;      // [n, 4] = (sequence, first row, rows, offset in the portion)
  int C, K;
  int add;               // 1: the input itself is added to the result
};

// Grid (tiles, channels / 256): 32 groups of eight channels times four groups of four rows.  Only the portion's first tile reads the
// state, so that tile also replaces it, after its own reads.  KT: taps known to the compiler (0: any number).
constexpr int GR_ROWS = GR_TILE / 4;
template <typename T, int KT>
__global__ void __launch_bounds__(GR_THREADS, sizeof(T) == 2 ? 5 : 4) causal_conv_kernel(const ConvParams p) {
  const int* tl = p.tiles + blockIdx.x * 4;
  const int s = tl[0], row0 = tl[1], rows = tl[2], off = tl[3], K = KT > 0 ? KT : p.K;
  const int c = (blockIdx.y * 32 + (threadIdx.x & 31)) * 8, t0 = (threadIdx.x >> 5) * GR_ROWS;
  const int slot = s < 0 ? -1 : p.slot[s];
  if (slot < 0 || rows <= 0) return;
  const bool fresh = p.start[s] == 0, in = c < p.C;
  const int cc = in ? c : 0;
  const T* x = static_cast<const T*>(p.x) + cc;
  const T* taps = static_cast<const T*>(p.taps) + static_cast<size_t>(cc) * K;
  float* st = p.state + (static_cast<size_t>(slot) * p.C + cc) * (K - 1);
  float xb[8] = {}, cb[8] = {};
  if (p.xb) vload8(static_cast<const T*>(p.xb) + cc, xb);
  if (p.cb) vload8(static_cast<const T*>(p.cb) + cc, cb);
  // Only the first rows of the first tile look back into the state.
  constexpr int KK = KT > 0 ? KT : 1, OLD = KT > 1 ? KT - 1 : 1;
  const bool head = off == 0 && t0 == 0;
  float w[KK * 8];                                   // a channel's taps are neighbours
  if constexpr (KT > 0) {
#pragma unroll
    for (int i = 0; i < KK; ++i) {
      float f[8];
      vload8(taps + i * 8, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) w[i * 8 + e] = f[e];
    }
  }
  // known taps: the state of these channels as it lies in memory, [channel][input]
  auto load_old = [&](float (&old)[OLD * 8]) {
    if constexpr (KT > 1) {
#pragma unroll
      for (int i = 0; i < OLD; ++i) {
        float f[8] = {};
        if (!fresh) vload8(st + i * 8, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) old[i * 8 + e] = f[e];
      }
    }
  };
  if constexpr (KT > 0) {
#pragma unroll
    for (int e = 0; e < 8; ++e) w[e * KT + KT - 1] += p.add ? 1.f : 0.f;
  }
  auto tap = [&](int e, int j) {                     // of channel e, j tokens back
    if constexpr (KT > 0) return w[e * KT + KT - 1 - j];
    else return to_f(taps[e * K + K - 1 - j]) + (j == 0 && p.add ? 1.f : 0.f);
  };
  auto input = [&](int at, float (&f)[8], const float (&old)[OLD * 8]) {          // input at index `at` of the portion
    if (at >= 0) {
      vload8(x + (static_cast<size_t>(row0) + at - off) * p.ld, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] += xb[e];
    } else if constexpr (KT > 1) {
#pragma unroll
      for (int j = 0; j < OLD; ++j)
        if (j == OLD + at)
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = old[e * OLD + j];
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = fresh ? 0.f : st[e * (K - 1) + K - 1 + at];
    }
  };
  T* dst = static_cast<T*>(p.u) + (static_cast<size_t>(row0) + t0) * p.C + c;
  if (in && t0 < rows) {
    const int n = min(GR_ROWS, rows - t0);
    if (KT > 0 && !head) {                           // all inputs are rows of this portion: requested together
      Packed8<T> raw[GR_ROWS + KK - 1];
#pragma unroll
      for (int i = 0; i < GR_ROWS + KK - 1; ++i) raw[i].load(x + (static_cast<size_t>(row0) + min(t0 + i - (KK - 1), rows - 1)) * p.ld);
#pragma unroll
      for (int o = 0; o < GR_ROWS; ++o) {
        if (o >= n) break;
        float acc[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = cb[e];
#pragma unroll
        for (int j = 0; j < KK; ++j) {
          float f[8];
          raw[o + KK - 1 - j].get(f);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[e] = fmaf(tap(e, j), f[e] + xb[e], acc[e]);
        }
        vstore8(dst + static_cast<size_t>(o) * p.C, acc);
      }
    } else if constexpr (KT > 0) {                   // the portion's first rows
      float old[OLD * 8];
      load_old(old);
#pragma unroll
      for (int o = 0; o < GR_ROWS; ++o) {
        if (o >= n) break;
        float acc[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = cb[e];
#pragma unroll
        for (int j = 0; j < KK; ++j) {
          float f[8];
          input(o - j, f, old);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[e] = fmaf(tap(e, j), f[e], acc[e]);
        }
        vstore8(dst + static_cast<size_t>(o) * p.C, acc);
      }
    } else {
      const float old[OLD * 8] = {};
      for (int o = 0; o < n; ++o) {
        float acc[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = cb[e];
        for (int j = 0; j < K; ++j) {
          float f[8];
          input(off + t0 + o - j, f, old);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[e] = fmaf(tap(e, j), f[e], acc[e]);
        }
        vstore8(dst + static_cast<size_t>(o) * p.C, acc);
      }
    }
  }
  if (off != 0 || K < 2) return;
  __syncthreads();
  if (!in || threadIdx.x >= 32) return;              // the warp of the first rows
  const int count = p.cu[s + 1] - p.cu[s];
  float old[OLD * 8];
  if constexpr (KT > 1) {
    load_old(old);
    float now[OLD * 8];
#pragma unroll
    for (int j = 0; j < OLD; ++j) {
      float f[8];
      input(count - OLD + j, f, old);
#pragma unroll
      for (int e = 0; e < 8; ++e) now[e * OLD + j] = f[e];
    }
#pragma unroll
    for (int i = 0; i < OLD; ++i) {
      float f[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = now[i * 8 + e];
      vstore8(st + i * 8, f);
    }
  } else {
    for (int j = 0; j < K - 1; ++j) {                // in this order an old input is read before its place is written
      float f[8];
      input(count - (K - 1) + j, f, old);
#pragma unroll
      for (int e = 0; e < 8; ++e) st[e * (K - 1) + j] = f[e];
    }
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
  float* ws;             // [runs, 2, C]: transfer (product, end state), then [.., 0, ..] the state at the run's start
  const int* cu;
  const int* start;
  const int* slot;
  const int* chunks;     // [n, 4], several runs each
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

constexpr int GR_RUN = 32;

// Rows of run h of a chunk.
__device__ __forceinline__ int run_rows(int rows, int h) { return max(0, min(GR_RUN, rows - h * GR_RUN)); }

template <typename T>
__global__ void __launch_bounds__(GR_THREADS) rec_transfer_kernel(const RecParams p) {
  const int* ch = p.chunks + (blockIdx.x >> 1) * 4;
  const int c = blockIdx.y * GR_THREADS + threadIdx.x, h = blockIdx.x & 1, n = run_rows(ch[2], h);
  if (c >= p.C || p.slot[ch[0]] < 0) return;
  const RecChannel<T> k(p, c);
  float A = 1.f, S = 0.f;
#pragma unroll 4
  for (int t = 0; t < n; ++t) {
    const float2 g = k.step(p, static_cast<size_t>(ch[1]) + h * GR_RUN + t);
    A *= g.x;
    S = fmaf(g.x, S, g.y);
  }
  float* w = p.ws + static_cast<size_t>(blockIdx.x) * 2 * p.C + c;
  w[0] = A;
  w[p.C] = S;
}

// Grid (channels, long sequences); per: runs of a chunk
__global__ void __launch_bounds__(GR_THREADS) rec_carry_kernel(const RecParams p, int per) {
  const int c = blockIdx.x * GR_THREADS + threadIdx.x, s = p.seq0 + blockIdx.y;
  const int slot = p.slot[s];
  if (c >= p.C || slot < 0) return;
  float* st = p.state + static_cast<size_t>(slot) * p.C + c;
  float S = p.start[s] == 0 ? 0.f : *st;
  const int c0 = p.first[blockIdx.y] * per, c1 = p.first[blockIdx.y + 1] * per;
  constexpr int U = 16;
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

// RUNS: grid (runs, channels), from the states rec_carry left; else grid (sequences, channels), from the slots and back to them.
template <typename T, bool RUNS>
__global__ void __launch_bounds__(GR_THREADS) rec_out_kernel(const RecParams p) {
  const int c = blockIdx.y * GR_THREADS + threadIdx.x;
  const int* ch = RUNS ? p.chunks + (blockIdx.x >> 1) * 4 : nullptr;
  const int s = RUNS ? ch[0] : p.seq0 + static_cast<int>(blockIdx.x);
  const int slot = p.slot[s];
  if (c >= p.C || slot < 0) return;
  const size_t row0 = RUNS ? ch[1] + (blockIdx.x & 1) * GR_RUN : p.cu[s];
  const int rows = RUNS ? run_rows(ch[2], blockIdx.x & 1) : p.cu[s + 1] - p.cu[s];
  float* st = p.state + static_cast<size_t>(slot) * p.C + c;
  float S = RUNS ? p.ws[static_cast<size_t>(blockIdx.x) * 2 * p.C + c] : p.start[s] == 0 ? 0.f : *st;
  const RecChannel<T> k(p, c);
#pragma unroll 4
  for (int t = 0; t < rows; ++t) {
    const size_t row = row0 + t;
    const float2 g = k.step(p, row);
    const float y = gelu_tanh_t<T>(to_f(static_cast<const T*>(p.y)[row * p.ld_y + c]) + k.yb);
    S = fmaf(g.x, S, g.y);
    static_cast<T*>(p.out)[row * p.ld_out + c] = from_f<T>(S * y);
  }
  if (!RUNS) *st = S;
}

// ---- both passes with their gates on the tensor cores ---------------------------------------------------------------------------
// A CTA keeps the two gates' weights of up to 128 channels of a block in shared memory (they read all of the block's channels of u)
// and walks chunks of 128 tokens.  Four warps per run of 32 tokens walk it, thread = channel; one more warp brings u by TMA (one chunk
// ahead, where there is room for two) and issues the products, those of the next chunk under the recurrence of this one.
constexpr int RG_CHUNK = 128, RG_RUNS = RG_CHUNK / GR_RUN, RG_WARPS = 4 * RG_RUNS, RG_THREADS = 32 * (RG_WARPS + 1);
constexpr int RG_MAX_BLOCK = 256;
constexpr int RG_TMEM = 512;           // two accumulators of two gates of a chunk: all of it, so one CTA per SM
typedef __nv_bfloat16 rg_bf16;

struct RecGateSmem {
  int kc, weights, stage, stages, total;       // 64-channel pieces of a block; bytes
  __host__ __device__ explicit RecGateSmem(int block) {
    kc = (block + 63) / 64;
    weights = 2 * kc * 128 * 128;
    stage = kc * RG_CHUNK * 128;
    stages = weights + 2 * stage <= 224 * 1024 ? 2 : 1;
    total = weights + stages * stage + 64 + 1024;
    if (total < 120 * 1024) total = 120 * 1024;       // more than half of an SM's
  }
};

__device__ __forceinline__ float sqrt_fast(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <bool OUT>
__global__ void __launch_bounds__(RG_THREADS, 1) rec_gates_kernel(const __grid_constant__ CUtensorMap tmU, const __grid_constant__ CUtensorMap tmW,
                                                                  const RecParams p, int nchunks, int tiles_per_block, int tile_channels, int* status) {
  extern __shared__ uint8_t rg_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rg_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const RecGateSmem L(p.block);
  uint8_t* su = sm + L.weights;
  uint64_t* bars = reinterpret_cast<uint64_t*>(su + L.stages * L.stage);
  uint64_t *w_full = bars, *u_full = bars + 1, *done = bars + 3, *used = bars + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 7);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, quarter = warp & 3, run = warp >> 2;
  const int b = blockIdx.x / tiles_per_block, c0 = blockIdx.x % tiles_per_block * tile_channels;     // first channel, in the block
  if (tid == 0) {
    for (int i = 0; i < 5; ++i) mbar_init(bars + i, 1);
    for (int i = 0; i < 2; ++i) mbar_init(used + i, RG_WARPS);
    mbar_fence_init();
  }
  if (warp == RG_WARPS) {
    tmem_alloc(tmem_slot, RG_TMEM);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(tmem_slot);
  const int stride = gridDim.y, mine = (nchunks - static_cast<int>(blockIdx.y) + stride - 1) / stride;      // chunks of this CTA
  auto chunk_of = [&](int it) { return static_cast<int>(blockIdx.y) + it * stride; };
  if (warp == RG_WARPS) {
    const bool leader = elect_one();
    auto load_u = [&](int it) {
      if (!leader) return;
      const int st = it % L.stages, row = p.chunks[chunk_of(it) * 4 + 1];
      mbar_expect_tx(u_full + st, L.stage);
      for (int k = 0; k < L.kc; ++k)
        tma_load_2d(su + st * L.stage + k * (RG_CHUNK * 128), &tmU, u_full + st, b * p.block + k * 64, row);
    };
    if (leader) {
      mbar_expect_tx(w_full, L.weights);
      for (int g = 0; g < 2; ++g)
        for (int k = 0; k < L.kc; ++k) tma_load_3d(sm + (g * L.kc + k) * 16384, &tmW, w_full, k * 64, c0, 2 * b + g);
    }
    for (int i = 0; i < L.stages && i < mine; ++i) load_u(i);
    mbar_wait_warp(w_full, 0, status, ERR_GEMM_MMA_WAIT_FULL);
    // Gates of chunk `it`: of its accumulator (256 columns, used again two chunks later) the first half is the recurrence gate's, the
    // second the input gate's.
    for (int it = 0; it < mine; ++it) {
      const int st = it % L.stages, next = it + 1;
      mbar_wait_warp(u_full + st, (it / L.stages) & 1, status, ERR_GEMM_MMA_WAIT_FULL);
      tc_fence_after();
      if (leader) {
        constexpr uint32_t idesc = make_idesc_f16(1, 128, RG_CHUNK, 0, 0);
        for (int g = 0; g < 2; ++g)
          for (int k = 0; k < L.kc; ++k) {
            const uint64_t da = make_smem_desc_sw128(smem_u32(sm + (g * L.kc + k) * 16384), 16, 1024),
                           db = make_smem_desc_sw128(smem_u32(su + st * L.stage + k * (RG_CHUNK * 128)), 16, 1024);
#pragma unroll
            for (int ks = 0; ks < 4; ++ks)
              umma_f16_ss(tmem + (it & 1) * (2 * RG_CHUNK) + g * RG_CHUNK, desc_advance(da, ks * 32), desc_advance(db, ks * 32), idesc,
                          k > 0 || ks > 0 ? 1u : 0u);
          }
        umma_commit(done + (it & 1));
      }
      __syncwarp();
      if (next >= L.stages && next < mine) {        // chunk `last` has been read: its stage, and the accumulator before this one
        const int last = next - L.stages;
        mbar_wait_warp(used + (last & 1), (last >> 1) & 1, status, ERR_GEMM_PRODUCER_WAIT);
        tc_fence_after();
        load_u(next);
      }
    }
  } else {
    const int l = quarter * 32 + lane;                // lane of the accumulator
    const bool in = l < tile_channels && c0 + l < p.block;
    const int c = in ? c0 + l : c0, ch = b * p.block + c;      // lanes without a channel read the tile's first one's
    const RecChannel<rg_bf16> K(p, ch);
    const uint32_t at = tmem + (static_cast<uint32_t>(quarter * 32) << 16) + run * GR_RUN;
    const int u_at = (c >> 6) * (RG_CHUNK * 128) + (c & 7) * 2, u_piece = (c >> 3) & 7;
    const bool idle = quarter * 32 >= tile_channels;  // the whole warp
    constexpr float LOG2E = 1.4426950408889634f;
    const float br2 = -LOG2E * K.br, bi2 = -LOG2E * K.bi, sp2 = -LOG2E * K.sp;
    for (int it = 0; it < mine; ++it) {
      const int st = it % L.stages, chunk = chunk_of(it);
      const int* cd = p.chunks + chunk * 4;
      const size_t row0 = cd[1] + run * GR_RUN;
      const int n = idle ? 0 : run_rows(cd[2], run);
      const size_t wi = (static_cast<size_t>(chunk) * RG_RUNS + run) * 2 * p.C + ch;
      float A = 1.f, S = 0.f;
      if (OUT) S = p.ws[wi];
      mbar_wait_warp(u_full + st, (it / L.stages) & 1, status, ERR_GEMM_MMA_WAIT_FULL);       // u itself is read below
      mbar_wait_warp(done + (it & 1), (it >> 1) & 1, status, ERR_GEMM_EPI_WAIT);
      tc_fence_after();
      const uint8_t* ut = su + st * L.stage + u_at;
      const rg_bf16* yp = OUT ? static_cast<const rg_bf16*>(p.y) + row0 * p.ld_y + ch : nullptr;
      rg_bf16* op = OUT ? static_cast<rg_bf16*>(p.out) + row0 * p.ld_out + ch : nullptr;
      // sixteen tokens from t0 on; WHOLE: all of them exist
      auto tokens = [&](auto whole, int t0) {
        constexpr bool WHOLE = decltype(whole)::value;
        uint32_t zr[16], zi[16];
        float y[16];
        if (OUT) {
#pragma unroll
          for (int i = 0; i < 16; ++i) y[i] = __bfloat162float(yp[(WHOLE ? t0 + i : min(t0 + i, n - 1)) * p.ld_y]);
        }
        tmem_ld_32x32b_x16(at + (it & 1) * (2 * RG_CHUNK) + t0, zr);
        tmem_ld_32x32b_x16(at + (it & 1) * (2 * RG_CHUNK) + RG_CHUNK + t0, zi);
        tmem_ld_wait();
        const uint8_t* ur = ut + (run * GR_RUN + t0) * 128;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float u = __bfloat162float(*reinterpret_cast<const rg_bf16*>(ur + i * 128 + ((u_piece ^ (i & 7)) << 4)));
          // both sigmoids with one reciprocal: 1 / (A B) gives 1 / A and 1 / B (the exponents are bounded so that A B stays finite)
          const float ea = 1.f + fast_exp2(fminf(fmaf(-LOG2E, __uint_as_float(zr[i]), br2), 62.f));
          const float eb = 1.f + fast_exp2(fminf(fmaf(-LOG2E, __uint_as_float(zi[i]), bi2), 62.f));
          const float q = __fdividef(1.f, ea * eb);
          const float x = sp2 * (eb * q);             // log2 a
          const float X = (2.f / LOG2E) * x;
          float a = fast_exp2(x);
          // 1 - a^2: where it cancels, the first terms of its series in X = 2 log a (relative error X^2 / 6)
          const float m = X > -0.01f ? -X * fmaf(0.5f, X, 1.f) : fmaf(-a, a, 1.f);
          float inc = sqrt_fast(m) * (ea * q) * u;
          if (!WHOLE && t0 + i >= n) {
            a = 1.f;
            inc = 0.f;
          }
          S = fmaf(a, S, inc);
          if (!OUT) A *= a;
          if (OUT && in && (WHOLE || t0 + i < n))
            op[static_cast<long long>(t0 + i) * p.ld_out] = __float2bfloat16(S * gelu_tanh_t<rg_bf16>(y[i] + K.yb));
        }
      };
#pragma unroll 1
      for (int t0 = 0; t0 < n; t0 += 16) {            // n is the same for the whole warp
        if (n - t0 >= 16) tokens(std::true_type{}, t0);
        else tokens(std::false_type{}, t0);
      }
      if (!OUT && in) {
        p.ws[wi] = A;
        p.ws[wi + p.C] = S;
      }
      tc_fence_before();
      mbar_arrive_warp(used + (it & 1));                         // this warp has read its part of the stage and of the accumulator
    }
  }
  if (*reinterpret_cast<volatile int*>(status) != 0) {     // copies and products in flight land before shared memory and TMEM go away
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == RG_WARPS) {
    tc_fence_after();
    tmem_dealloc(tmem, RG_TMEM);
  }
}

template <bool OUT>
static int launch_gates(const CUtensorMap* tu, const CUtensorMap* tw, const RecParams& p, int nchunks, cudaStream_t stream) {
  auto kern = rec_gates_kernel<OUT>;
  int* status = status_ptr();
  if (!status) return 3;
  const RecGateSmem L(p.block);
  static int set[64] = {0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (set[dev & 63] < L.total) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total) != cudaSuccess) {
      set_error("rec_gates: cannot set shared memory size (%d)", L.total);
      return 1;
    }
    set[dev & 63] = L.total;
  }
  // tiles of equal size, in whole warps where that costs none of them
  const int per = (p.block + 127) / 128, x = p.C / p.block * per;
  int tile = (p.block + per - 1) / per, y = num_sms() / x;
  if ((tile + 31) / 32 * 32 * (per - 1) < p.block) tile = (tile + 31) / 32 * 32;
  if (y < 1) y = 1;
  if (y > nchunks) y = nchunks;
  kern<<<dim3(x, y), RG_THREADS, L.total, stream>>>(*tu, *tw, p, nchunks, per, tile, status);
  B2_CHECK_LAUNCH("rec_gates");
  return 0;
}

}  // namespace b2

using namespace b2;

B2_EXPORT int b2_causal_conv(const void* x, long long ld, const void* xb, const void* taps, const void* cb, float* state, void* u,
                             const int* cu, const int* start, const int* slot, const int* tiles, int ntiles, int C, int K,
                             int add, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (ntiles <= 0) return 0;
  if (C < 8 || C % 8 || ld % 8 || K < 1 || K - 1 > GR_TILE) {
    set_error("causal_conv: channels in multiples of 8 and 1 to %d taps required", GR_TILE + 1);
    return 10;
  }
  const ConvParams p = {x, ld, xb, taps, cb, state, u, cu, start, slot, tiles, C, K, add};
  const dim3 grid(ntiles, (C / 8 + 31) / 32);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (K == 4) {
    B2_DISPATCH_T(is_f32, (causal_conv_kernel<T, 4><<<grid, GR_THREADS, 0, st>>>(p)););
  } else {
    B2_DISPATCH_T(is_f32, (causal_conv_kernel<T, 0><<<grid, GR_THREADS, 0, st>>>(p)););
  }
  B2_CHECK_LAUNCH("causal_conv");
  return 0;
}

// Sequences seq0 .. seq0 + nseq - 1; nchunks > 0: they are long, chunks / first describe them and ws is fp32 [nchunks, 2, 2, C].
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
    B2_DISPATCH_T(is_f32, rec_transfer_kernel<T><<<dim3(2 * nchunks, cy), GR_THREADS, 0, st>>>(p););
    B2_CHECK_LAUNCH("rec_transfer");
    rec_carry_kernel<<<dim3(cy, nseq), GR_THREADS, 0, st>>>(p, 2);
    B2_CHECK_LAUNCH("rec_carry");
    B2_DISPATCH_T(is_f32, (rec_out_kernel<T, true><<<dim3(2 * nchunks, cy), GR_THREADS, 0, st>>>(p)););
  } else {
    B2_DISPATCH_T(is_f32, (rec_out_kernel<T, false><<<dim3(nseq, cy), GR_THREADS, 0, st>>>(p)););
  }
  B2_CHECK_LAUNCH("linear_recurrence");
  return 0;
}

// Long sequences in bf16 with the gates' products inside: u [M, C] contiguous, w [C / block, 2, block, block], blocks up to 256
// channels in multiples of 8; chunks of 128 rows, ws fp32 [nchunks, 4, 2, C].
B2_EXPORT int b2_gated_recurrence(const void* u, const void* w, const void* zb, const void* lam, const void* y, long long ld_y,
                                  const void* yb, void* out, long long ld_out, float* state, float* ws, const int* start, const int* slot,
                                  const int* chunks, const int* first, int nchunks, int seq0, int nseq, int M, int C, int block,
                                  void* stream) {
  b2::ensure_thread_context();
  if (nseq <= 0 || nchunks <= 0) return 0;
  if (block < 8 || block % 8 || block > RG_MAX_BLOCK || C < block || C % block || nseq > 65535) {
    set_error("gated_recurrence: blocks up to %d channels in multiples of 8 required", RG_MAX_BLOCK);
    return 10;
  }
  const RecParams p = {u, nullptr, zb, lam, y, yb, out, state, ws, nullptr, start, slot, chunks, first, C, 0, ld_y, ld_out, C, block, seq0};
  const uint64_t n = block, dims[3] = {n, n, 2ull * (C / block)}, strides[2] = {2 * n, 2 * n * n};
  const uint32_t box[3] = {64, 128, 1};
  const CUtensorMap *tw = tensor_map_nd_bf16(w, 3, dims, strides, box, 3), *tu = tensor_map_2d_bf16(u, M, C, C, RG_CHUNK, 64);
  if (!tw || !tu) return 2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (const int rc = launch_gates<false>(tu, tw, p, nchunks, st)) return rc;
  rec_carry_kernel<<<dim3((C + GR_THREADS - 1) / GR_THREADS, nseq), GR_THREADS, 0, st>>>(p, RG_RUNS);
  B2_CHECK_LAUNCH("rec_carry");
  return launch_gates<true>(tu, tw, p, nchunks, st);
}
