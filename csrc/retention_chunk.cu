// Retention and matrix memory over long prompt portions, chunk by chunk (RET_C tokens), in three launches per layer:
//
//   1. every chunk's own contribution to the state, K^T V with the decays to the chunk's end       (all chunks at once)
//   2. the running state at every chunk's start: S_c = a^n S_{c-1} + contribution                   (a scan, element-wise)
//   3. o = a^{t+1} S_c^T q + sum_{j <= t} a^{t-j} (q . k_j) v_j, per-head norm, gate, store         (all chunks at once)
//      (or, for heads that are normed together, weight, sigmoid gate, store and each head's sum of squares)
//
// Matrix memory (MEM) weighs token j for a later token t by exp(b_t - b_j + i_j - m_t), b the running sum of the log forget gates.
// With g_j = i_j - b_j and M_t = max(m_0, max_{j <= t} g_j), b and m counted from the chunk's start: m_t = b_t + M_t, the weight is
// exp(g_j - M_t), that of the state before the chunk exp(m_0 - M_t), and none of them is above one.  Contributions are kept
// relative to the chunk's own largest g; the scan carries m along and rescales.  The normaliser is the row sum of the weighted
// scores plus the query's product with the carried n.
//
// The products are tcgen05 MMAs of one 128-token tile with fp32 accumulators in TMEM.  An fp32 operand that enters the
// recurrence or weighs a value (k, the state, the weights) is the sum of two bf16 numbers, hi + lo, and takes two MMAs;
// v is exact in bf16, and q, which enters no recurrence, is rounded to bf16.  The operands are computed on the way in
// (rotation, decays, split), so the threads write the 128-byte-swizzled tiles themselves instead of TMA.
#include "host.h"
#include "mma_split.cuh"
#include "vec.cuh"

namespace b2 {

constexpr int RET_C = 128;
constexpr int RET_THREADS = 256;
constexpr float MEMORY_EPS = 1e-6f;
typedef __nv_bfloat16 bf16_t;

struct RetParams {
  const bf16_t* q;
  const bf16_t* k;
  const bf16_t* v;
  const bf16_t* gate;
  bf16_t* out;
  float* ws;            // [chunks, H, dkp, dvp]
  float* state;         // [slots, H, dkp, dvp]
  const float* decay;
  const float* cs;      // [M, rot / 2]
  const float* sn;
  const int* chunks;    // [n, 4] = (sequence, first row, rows, offset in the portion)
  const int* first;     // [nlong + 1] first chunk of each long sequence
  const int* start;     // [nseq]
  const int* slot;      // [nseq]
  const bf16_t* norm_w; // joint norm: [H * dvp]
  float* joint_ss;      // [M, H] sums of squares for the reader, or null: a norm per head and a silu gate
  long long ld_in, ld_out;
  int H, dk, dkp, dv, dvp, rot, seq0;
  float kscale, eps;
  // matrix memory: gates before bias and cap [M, ld_z] and their biases [H]; normaliser and maximum per slot; per chunk and head the
  // contribution to n [dkp], (sum of log forget gates, largest g), and the maximum at the chunk's start
  const float* zi;
  const float* zf;
  const bf16_t* bi;
  const bf16_t* bf;
  float* n;              // [slots, H, dkp]
  float* m;              // [slots, H]
  float* wn;
  float2* wg;
  float* wm;
  long long ld_z;
  float cap, qscale, oscale;
};

__device__ __forceinline__ float ret_pow(float l2a, int n) { return n == 0 ? 1.f : fast_exp2(l2a * n); }

// Swizzled bf16 tile: halves of 64 columns, each [rows x 128 bytes]; `c` is a multiple of 8.
__device__ __forceinline__ uint8_t* ret_at(uint8_t* tile, int half_bytes, int row, int c) {
  return tile + (c >> 6) * half_bytes + row * 128 + ((((c >> 3) & 7) ^ (row & 7)) << 4);
}
template <bool LO>
__device__ __forceinline__ void ret_put(uint8_t* hi, uint8_t* lo, int half_bytes, int row, int c, const float (&f)[8]) {
  bf16_t* h = reinterpret_cast<bf16_t*>(ret_at(hi, half_bytes, row, c));
  if (LO) store8_split(h, reinterpret_cast<bf16_t*>(ret_at(lo, half_bytes, row, c)), f);
  else vstore8(h, f);
}

// ROWS rows of one head, rotated, times scale(t), as hi (and lo) tiles `width` (64 or 128) columns wide; zero past `n` rows
// and dkp channels.
template <int ROWS, bool LO, typename F>
__device__ __forceinline__ void ret_load_rotated(uint8_t* hi, uint8_t* lo, int width, const bf16_t* src, size_t row0, int n,
                                                 const RetParams& p, F scale) {
  const int half = p.rot / 2, tid = threadIdx.x;
  if (half % 8 == 0) {
    // Rotated pairs of 8-channel pieces, then plain pieces.  Two items at a time, their loads unconditional (clamped to rows
    // and channels that exist, the result dropped), so that all of them are in flight together.
    const int rv = half / 8, pieces = rv + (width - p.rot) / 8, total = ROWS * pieces;
    for (int i0 = tid; i0 < total; i0 += 2 * RET_THREADS) {
      uint4 u4[2], w4[2];
      float4 c4[2][2], s4[2][2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int i = min(i0 + k * RET_THREADS, total - 1), t = min(i / pieces, n - 1), c = i % pieces;
        const int at = c < rv ? c * 8 : min(p.rot + (c - rv) * 8, p.dkp - 8);
        const bf16_t* s = src + (row0 + t) * p.ld_in + at;
        u4[k] = *reinterpret_cast<const uint4*>(s);
        w4[k] = *reinterpret_cast<const uint4*>(c < rv ? s + half : s);
        if (rv > 0) {
          const size_t f = (row0 + t) * half + (c < rv ? c * 8 : 0);
          c4[k][0] = *reinterpret_cast<const float4*>(p.cs + f);
          c4[k][1] = *reinterpret_cast<const float4*>(p.cs + f + 4);
          s4[k][0] = *reinterpret_cast<const float4*>(p.sn + f);
          s4[k][1] = *reinterpret_cast<const float4*>(p.sn + f + 4);
        }
      }
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int i = i0 + k * RET_THREADS, t = i / pieces, c = i % pieces;
        if (i >= total) break;
        float u[8], x[8], y[8];
        unpack8(u4[k], u);
        if (c < rv) {
          const float f = t < n ? scale(t) : 0.f;
          float w[8];
          unpack8(w4[k], w);
          const float cs[8] = {c4[k][0].x, c4[k][0].y, c4[k][0].z, c4[k][0].w, c4[k][1].x, c4[k][1].y, c4[k][1].z, c4[k][1].w};
          const float sn[8] = {s4[k][0].x, s4[k][0].y, s4[k][0].z, s4[k][0].w, s4[k][1].x, s4[k][1].y, s4[k][1].z, s4[k][1].w};
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            x[e] = (u[e] * cs[e] - w[e] * sn[e]) * f;
            y[e] = (w[e] * cs[e] + u[e] * sn[e]) * f;
          }
          ret_put<LO>(hi, lo, ROWS * 128, t, c * 8, x);
          ret_put<LO>(hi, lo, ROWS * 128, t, half + c * 8, y);
        } else {
          const int at = p.rot + (c - rv) * 8;
          const float f = t < n && at < p.dkp ? scale(t) : 0.f;
#pragma unroll
          for (int e = 0; e < 8; ++e) u[e] = f != 0.f ? u[e] * f : 0.f;
          ret_put<LO>(hi, lo, ROWS * 128, t, at, u);
        }
      }
    }
    return;
  }
  for (int i = tid; i < ROWS * (width / 8); i += RET_THREADS) {
    const int t = i / (width / 8), c8 = i % (width / 8) * 8;
    float x[8] = {};
    if (t < n && c8 < p.dkp) {
      const bf16_t* s = src + (row0 + t) * p.ld_in;
      const float fs = scale(t);
      for (int e = 0; e < 8; ++e) {
        const int c = c8 + e;
        x[e] = to_f(s[c]);
        if (c < p.rot) {
          const int f = c < half ? c : c - half;
          const float o = to_f(s[c < half ? c + half : c - half]);
          x[e] = x[e] * p.cs[(row0 + t) * half + f] + (c < half ? -o : o) * p.sn[(row0 + t) * half + f];
        }
        x[e] *= fs;
      }
    }
    ret_put<LO>(hi, lo, ROWS * 128, t, c8, x);
  }
}

__device__ __forceinline__ void ret_load_v(uint8_t* tile, int width, const bf16_t* src, size_t row0, int n, const RetParams& p) {
  const int pieces = width / 8;                    // RET_C * pieces is a multiple of 4 * RET_THREADS
  for (int i0 = threadIdx.x; i0 < RET_C * pieces; i0 += 4 * RET_THREADS) {
    uint4 u[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = i0 + k * RET_THREADS, t = min(i / pieces, n - 1), c = min(i % pieces * 8, p.dvp - 8);
      u[k] = *reinterpret_cast<const uint4*>(src + (row0 + t) * p.ld_in + c);
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = i0 + k * RET_THREADS, t = i / pieces, c = i % pieces * 8;
      *reinterpret_cast<uint4*>(ret_at(tile, RET_C * 128, t, c)) = t < n && c < p.dvp ? u[k] : make_uint4(0, 0, 0, 0);
    }
  }
}

constexpr int RET_TILE = RET_C * 128 * 2;        // a full [128 x 128] bf16 tile: 32 KiB
constexpr int RET_HALF = RET_C * 128;
// after the tiles: barrier and TMEM address (64 bytes), row sums (1 KiB, ret_out), matrix memory: gates, (ret_out) the carried n and
// row sums of the weights
constexpr int RET_GATES = 3 * RET_C * 4 + 32;
constexpr int RET_CONTRIB_BYTES = 3 * RET_TILE + 64 + 1024, MEM_CONTRIB_BYTES = RET_CONTRIB_BYTES + RET_GATES;
constexpr int RET_OUT_BYTES = 3 * RET_TILE + 64 + 1024 + 1024, MEM_OUT_BYTES = RET_OUT_BYTES + RET_GATES + 512 + 1024;

__device__ __forceinline__ uint8_t* ret_align(uint8_t* p) {
  return reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(p) + 1023) & ~static_cast<uintptr_t>(1023));
}

// The CTA's barrier and TMEM.  A wait that runs out sets the status word and lets everyone run on to the end (later waits
// return at once), so TMEM is always freed.
struct RetMma {
  uint64_t* bar;
  uint32_t* slot;
  int* status;
  uint32_t phase = 0, tmem = 0;
  __device__ __forceinline__ void setup(uint8_t* at, int* st, uint32_t cols) {
    bar = reinterpret_cast<uint64_t*>(at);
    slot = reinterpret_cast<uint32_t*>(at + 16);
    status = st;
    if (threadIdx.x == 0) {
      mbar_init(bar, 1);
      mbar_fence_init();
    }
    if (threadIdx.x < 32) {
      tmem_alloc(slot, cols);
      tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    tmem = *reinterpret_cast<volatile uint32_t*>(slot);
  }
  // operand tiles have been written by all threads: make them visible to the tensor core, then let warp 0 issue
  __device__ __forceinline__ void publish() {
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
  }
  __device__ __forceinline__ void wait() {
    mbar_wait_warp(bar, phase, status, ERR_ATTN_WAIT);
    phase ^= 1;
    tc_fence_after();
  }
  __device__ __forceinline__ void release(uint32_t cols) {
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x < 32) {
      tc_fence_after();
      tmem_dealloc(tmem, cols);
    }
  }
};

// Gates of a chunk's tokens: g, M (from m0 on) and b of the comment at the top, into shared memory; g is -inf past the n tokens.
struct RetGates {
  float g[RET_C], M[RET_C], b[RET_C], red[8];
};
static_assert(sizeof(RetGates) == RET_GATES, "shared memory of the gates");
__device__ __forceinline__ void ret_gates(const RetParams& p, int h, size_t row0, int n, float m0, RetGates& s) {
  const int t = threadIdx.x, warp = t >> 5, lane = t & 31;
  float i = -INFINITY, b = 0.f;
  if (t < n) {
    const float zf = p.zf[(row0 + t) * p.ld_z + h] + to_f(p.bf[h]), zi = p.zi[(row0 + t) * p.ld_z + h] + to_f(p.bi[h]);
    const float x = p.cap * tanhf(zf / p.cap);
    b = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
    i = p.cap * tanhf(zi / p.cap);
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float v = __shfl_up_sync(0xffffffffu, b, o);
    if (lane >= o) b += v;
  }
  if (lane == 31 && t < RET_C) s.red[warp] = b;
  __syncthreads();
  float g = -INFINITY, mx = -INFINITY;
  if (t < RET_C) {
    for (int w = 0; w < warp; ++w) b += s.red[w];
    if (t < n) g = i - b;
    mx = g;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, mx, o);
      if (lane >= o) mx = fmaxf(mx, v);
    }
    if (lane == 31) s.red[4 + warp] = mx;
  }
  __syncthreads();
  if (t < RET_C) {
    for (int w = 0; w < warp; ++w) mx = fmaxf(mx, s.red[4 + w]);
    s.g[t] = g;
    s.M[t] = fmaxf(mx, m0);
    s.b[t] = b;
  }
  __syncthreads();
}

template <bool MEM>
__global__ void __launch_bounds__(RET_THREADS, 2) ret_contrib_kernel(const RetParams p, int* status) {
  extern __shared__ uint8_t sm_raw[];
  uint8_t* sm = ret_align(sm_raw);
  uint8_t *sKh = sm, *sKl = sm + RET_TILE, *sV = sm + 2 * RET_TILE;
  RetGates& gates = *reinterpret_cast<RetGates*>(sm + 3 * RET_TILE + 64);
  RetMma mma;
  mma.setup(sm + 3 * RET_TILE, status, 128);
  const int* ch = p.chunks + blockIdx.x * 4;
  const int h = blockIdx.y, n = ch[2];
  const size_t row0 = ch[1];
  const float l2a = MEM ? 0.f : log2f(p.decay[h]);
  const int wk = p.dkp > 64 ? 128 : 64, wv = p.dvp > 64 ? 128 : 64;
  float top = 0.f;
  if (MEM) {
    ret_gates(p, h, row0, n, -INFINITY, gates);
    top = gates.M[RET_C - 1];
    if (threadIdx.x == 0) p.wg[static_cast<size_t>(blockIdx.x) * p.H + h] = make_float2(gates.b[RET_C - 1], top);
  }
  ret_load_rotated<RET_C, true>(sKh, sKl, wk, p.k + static_cast<size_t>(h) * p.dkp, row0, n, p,
                                [&](int t) { return MEM ? expf(gates.g[t] - top) : p.kscale * ret_pow(l2a, n - 1 - t); });
  ret_load_v(sV, wv, p.v + static_cast<size_t>(h) * p.dvp, row0, n, p);
  mma.publish();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) {
    // D[key channel, value channel]: both operands have the contraction (tokens) along the rows.  With 64 key channels the
    // accumulator's upper rows come from whatever follows the tile; they are not stored.
    const bool leader = elect_one();
    const uint32_t idesc = make_idesc_f16(1, 128, wv, 1, 1);
    const uint64_t dh = make_smem_desc_sw128(smem_u32(sKh), RET_HALF, 1024), dl = make_smem_desc_sw128(smem_u32(sKl), RET_HALF, 1024),
                   dv = make_smem_desc_sw128(smem_u32(sV), RET_HALF, 1024);
    if (leader) {
#pragma unroll
      for (int ks = 0; ks < RET_C / 16; ++ks) {
        umma_f16_ss(mma.tmem, desc_advance(dh, ks * 2048), desc_advance(dv, ks * 2048), idesc, ks != 0);
        umma_f16_ss(mma.tmem, desc_advance(dl, ks * 2048), desc_advance(dv, ks * 2048), idesc, 1);
      }
      umma_commit(mma.bar);
    }
    __syncwarp();
  }
  if (MEM) {                                       // the weighted keys' sum, two threads a channel; the second half by way of shared memory
    const int c = threadIdx.x & 127, t0 = (threadIdx.x >> 7) * 64;
    float s = 0.f;
    if (c < p.dkp)
      for (int t = t0; t < min(t0 + 64, n); ++t) {
        const int at = c & ~7;
        s += to_f(reinterpret_cast<const bf16_t*>(ret_at(sKh, RET_HALF, t, at))[c & 7]) +
             to_f(reinterpret_cast<const bf16_t*>(ret_at(sKl, RET_HALF, t, at))[c & 7]);
      }
    if (t0 > 0) gates.M[c] = s;
    __syncthreads();
    if (t0 == 0 && c < p.dkp) p.wn[(static_cast<size_t>(blockIdx.x) * p.H + h) * p.dkp + c] = s + gates.M[c];
  }
  mma.wait();
  const int quarter = warp & 3, half = warp >> 2, i0 = quarter * 32;
  float* w = p.ws + (static_cast<size_t>(blockIdx.x) * p.H + h) * p.dkp * p.dvp;
  uint8_t* stage = sm + warp * 4096;              // the operands have been read
#pragma unroll
  for (int c32 = 0; c32 < 2; ++c32) {
    const int c0 = half * 64 + c32 * 32;
    if (c0 >= wv) break;
    uint32_t t[32];
    tmem_ld_32x32b_x32(mma.tmem + (static_cast<uint32_t>(i0) << 16) + c0, t);
    tmem_ld_wait();
    uint4 v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = make_uint4(t[4 * j], t[4 * j + 1], t[4 * j + 2], t[4 * j + 3]);
    warp_store_rows_128B(stage, v, [&](int row) -> uint8_t* {
      if (i0 + row >= p.dkp || c0 + (lane & 7) * 4 >= p.dvp) return nullptr;
      return reinterpret_cast<uint8_t*>(w + static_cast<size_t>(i0 + row) * p.dvp + c0);
    });
  }
  mma.release(128);
}

// The same scan for matrix memory: the normaliser is dkp more elements of the state, and every thread carries the maximum (whose slot
// is only read here; ret_out replaces it).
__global__ void __launch_bounds__(256) mem_scan_kernel(const RetParams p) {
  const int h = blockIdx.y, s = p.seq0 + blockIdx.z;
  const int size = p.dkp * p.dvp, i = (blockIdx.x * 256 + threadIdx.x) * 4;
  const int slot = p.slot[s];
  if (i >= size + p.dkp || slot < 0) return;
  const size_t head = static_cast<size_t>(slot) * p.H + h;
  const bool fresh = p.start[s] == 0, mat = i < size;
  float* st = mat ? p.state + head * size + i : p.n + head * p.dkp + i - size;
  float4 S = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st);
  float m = fresh ? 0.f : p.m[head];
  const int c0 = p.first[blockIdx.z], c1 = p.first[blockIdx.z + 1];
  const size_t step = static_cast<size_t>(p.H) * (mat ? size : p.dkp);
  float* w = mat ? p.ws + (static_cast<size_t>(c0) * p.H + h) * size + i : p.wn + (static_cast<size_t>(c0) * p.H + h) * p.dkp + i - size;
  constexpr int U = 8;
  for (int c = c0; c < c1; c += U) {
    float4 kv[U];
    float2 g[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int at = min(u, c1 - 1 - c);
      kv[u] = *reinterpret_cast<const float4*>(w + at * step);
      g[u] = p.wg[static_cast<size_t>(c + at) * p.H + h];
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u >= c1) break;
      *reinterpret_cast<float4*>(w + u * step) = S;
      if (i == 0) p.wm[static_cast<size_t>(c + u) * p.H + h] = m;
      const float M = fmaxf(m, g[u].y), a = expf(m - M), b = expf(g[u].y - M);
      m = g[u].x + M;
      S.x = fmaf(a, S.x, b * kv[u].x);
      S.y = fmaf(a, S.y, b * kv[u].y);
      S.z = fmaf(a, S.z, b * kv[u].z);
      S.w = fmaf(a, S.w, b * kv[u].w);
    }
    w += U * step;
  }
  *reinterpret_cast<float4*>(st) = S;
}

// ws[c] <- state at the start of chunk c; the final state goes to the slot.  Grid (pieces of the state, H, long sequences).
__global__ void __launch_bounds__(256) ret_scan_kernel(const RetParams p) {
  const int h = blockIdx.y, s = p.seq0 + blockIdx.z;
  const int size = p.dkp * p.dvp, i = (blockIdx.x * 256 + threadIdx.x) * 4;
  const int slot = p.slot[s];
  if (i >= size || slot < 0) return;
  const float l2a = log2f(p.decay[h]);
  float* st = p.state + (static_cast<size_t>(slot) * p.H + h) * size + i;
  float4 S = p.start[s] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st);
  const int c0 = p.first[blockIdx.z], c1 = p.first[blockIdx.z + 1];
  const float full = exp2f(l2a * RET_C);
  const size_t step = static_cast<size_t>(p.H) * size;
  float* w = p.ws + (static_cast<size_t>(c0) * p.H + h) * size + i;
  constexpr int U = 8;
  for (int c = c0; c < c1; c += U) {
    float4 kv[U];
#pragma unroll
    for (int u = 0; u < U; ++u) kv[u] = *reinterpret_cast<const float4*>(w + min(u, c1 - 1 - c) * step);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u >= c1) break;
      *reinterpret_cast<float4*>(w + u * step) = S;
      const float a = c + u + 1 < c1 ? full : exp2f(l2a * p.chunks[(c + u) * 4 + 2]);   // only the last chunk may be short
      S.x = fmaf(a, S.x, kv[u].x);
      S.y = fmaf(a, S.y, kv[u].y);
      S.z = fmaf(a, S.z, kv[u].z);
      S.w = fmaf(a, S.w, kv[u].w);
    }
    w += U * step;
  }
  *reinterpret_cast<float4*>(st) = S;
}

// TMEM: columns 0..127 hold the weights' fp32 scores and then, as bf16 pairs, their hi (64) and lo (64) parts; 128..255 hold o.
// The state and the keys pass through one 32 KiB buffer in pieces of 64 rows, so that two CTAs fit on an SM and one's loads
// run under the other's products.
constexpr int RET_PIECE = 64;

template <bool MEM>
__global__ void __launch_bounds__(RET_THREADS, 2) ret_out_kernel(const RetParams p, int* status) {
  extern __shared__ uint8_t sm_raw[];
  uint8_t* sm = ret_align(sm_raw);
  uint8_t *sQ = sm, *sV = sm + RET_TILE, *hi = sm + 2 * RET_TILE, *lo = hi + RET_TILE / 2;
  float* xchg = reinterpret_cast<float*>(sm + 3 * RET_TILE + 64);     // [2 column halves][128 rows]
  RetMma mma;
  mma.setup(sm + 3 * RET_TILE, status, 256);
  const int* ch = p.chunks + blockIdx.x * 4;
  const int h = blockIdx.y, s = ch[0], n = ch[2];
  const size_t row0 = ch[1];
  const bool zero = ch[3] == 0 && p.start[s] == 0;       // nothing before this chunk
  const float l2a = MEM ? 0.f : log2f(p.decay[h]);
  RetGates& gates = *reinterpret_cast<RetGates*>(sm + 3 * RET_TILE + 64 + 1024);
  float* sn0 = reinterpret_cast<float*>(sm + 3 * RET_TILE + 64 + 1024 + RET_GATES);      // [128]
  float* swsum = sn0 + 128;                              // [2 column halves][128 rows]
  constexpr float LOG2E = 1.4426950408889634f;
  float m0 = 0.f;
  if (MEM) {
    m0 = p.wm[static_cast<size_t>(blockIdx.x) * p.H + h];
    ret_gates(p, h, row0, n, m0, gates);
    if (threadIdx.x < 128)
      sn0[threadIdx.x] = !zero && static_cast<int>(threadIdx.x) < p.dkp ? p.wn[(static_cast<size_t>(blockIdx.x) * p.H + h) * p.dkp + threadIdx.x] : 0.f;
    // the last chunk of a sequence leaves its maximum
    if (threadIdx.x == 0 && (blockIdx.x + 1 == gridDim.x || p.chunks[(blockIdx.x + 1) * 4] != s) && p.slot[s] >= 0)
      p.m[static_cast<size_t>(p.slot[s]) * p.H + h] = gates.b[n - 1] + gates.M[n - 1];
  }
  const int wk = p.dkp > 64 ? 128 : 64, wv = p.dvp > 64 ? 128 : 64;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quarter = warp & 3, half = warp >> 2;
  const int r = quarter * 32 + lane;                     // token of this thread, shared with the warp four further on
  const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
  const uint32_t tS = mma.tmem, tO = mma.tmem + 128;
  const bool mine = half * 64 < wv;                      // this thread has columns of o
  ret_load_rotated<RET_C, false>(sQ, nullptr, wk, p.q + static_cast<size_t>(h) * p.dkp, row0, n, p, [](int) { return 1.f; });
  ret_load_v(sV, wv, p.v + static_cast<size_t>(h) * p.dvp, row0, n, p);
  const bool leader = warp == 0 && elect_one();
  const uint64_t dq = make_smem_desc_sw128(smem_u32(sQ), 16, 1024);
  const uint32_t idesc_o = make_idesc_f16(1, 128, wv, 0, 1);
  float wsum = 0.f;                                      // matrix memory: this thread's part of n . q

  if (!zero) {
    const float* w = p.ws + (static_cast<size_t>(blockIdx.x) * p.H + h) * p.dkp * p.dvp;
    const int pieces = wv / 8;
    for (int r0 = 0; r0 < wk; r0 += RET_PIECE) {
      if (r0 > 0) mma.wait();
      for (int i0 = threadIdx.x; i0 < RET_PIECE * pieces; i0 += 2 * RET_THREADS) {   // a multiple of 2 * RET_THREADS
        float x[2][8];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const int i = i0 + k * RET_THREADS, t = min(r0 + i / pieces, p.dkp - 1), c = min(i % pieces * 8, p.dvp - 8);
          vload8(w + static_cast<size_t>(t) * p.dvp + c, x[k]);
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const int i = i0 + k * RET_THREADS, t = i / pieces, c = i % pieces * 8;
          const bool in = r0 + t < p.dkp && c < p.dvp;
#pragma unroll
          for (int e = 0; e < 8; ++e) x[k][e] = in ? x[k][e] : 0.f;
          ret_put<true>(hi, lo, RET_PIECE * 128, t, c, x[k]);
        }
      }
      mma.publish();
      if (leader) {
        const uint64_t dh = make_smem_desc_sw128(smem_u32(hi), RET_PIECE * 128, 1024),
                       dl = make_smem_desc_sw128(smem_u32(lo), RET_PIECE * 128, 1024);
#pragma unroll
        for (int ks = 0; ks < RET_PIECE / 16; ++ks) {
          const uint64_t a = desc_advance(dq, (r0 >> 6) * RET_HALF + ks * 32);
          umma_f16_ss(tO, a, desc_advance(dh, ks * 2048), idesc_o, r0 > 0 || ks > 0);
          umma_f16_ss(tO, a, desc_advance(dl, ks * 2048), idesc_o, 1);
        }
        umma_commit(mma.bar);
      }
      __syncwarp();
    }
    mma.wait();
    if (MEM) {                                           // this thread's half of q . n
      float d = 0.f;
      if (half * 64 < wk)
#pragma unroll
        for (int c = 0; c < 64; c += 8) {
          float q[8];
          vload8(reinterpret_cast<const bf16_t*>(ret_at(sQ, RET_HALF, r, half * 64 + c)), q);
#pragma unroll
          for (int e = 0; e < 8; ++e) d = fmaf(q[e], sn0[half * 64 + c + e], d);
        }
      wsum = d * fast_exp2((m0 - gates.M[r]) * LOG2E) * p.qscale;
    }
    if (mine) {                                          // o = a^{t+1} (q S)
      const float f = MEM ? fast_exp2((m0 - gates.M[r]) * LOG2E) * p.qscale : ret_pow(l2a, r + 1);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t t[16];
        tmem_ld_32x32b_x16(tO + lane_off + half * 64 + c * 16, t);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) t[i] = __float_as_uint(__uint_as_float(t[i]) * f);
        tmem_st_32x32b_x16(tO + lane_off + half * 64 + c * 16, t);
      }
      tmem_st_wait();
    }
  }
  for (int k0 = 0; k0 < n; k0 += RET_PIECE) {
    ret_load_rotated<RET_PIECE, true>(hi, lo, wk, p.k + static_cast<size_t>(h) * p.dkp, row0 + k0, n - k0, p,
                                      [&](int) { return p.kscale; });
    mma.publish();
    if (leader) {
      const uint32_t idesc = make_idesc_f16(1, 128, RET_PIECE, 0, 0);
      const uint64_t dh = make_smem_desc_sw128(smem_u32(hi), 16, 1024), dl = make_smem_desc_sw128(smem_u32(lo), 16, 1024);
      for (int ks = 0; ks < wk / 16; ++ks) {
        const uint64_t a = desc_advance(dq, (ks >> 2) * RET_HALF + (ks & 3) * 32);
        const uint32_t b = (ks >> 2) * (RET_PIECE * 128) + (ks & 3) * 32;
        umma_f16_ss(tS + k0, a, desc_advance(dh, b), idesc, ks != 0);
        umma_f16_ss(tS + k0, a, desc_advance(dl, b), idesc, 1);
      }
      umma_commit(mma.bar);
    }
    __syncwarp();
    mma.wait();
  }
  {
    // weights of this thread's 64 keys: decayed, causal, split
    uint32_t ph[32], pl[32];
    const float mr = MEM ? gates.M[r] : 0.f;
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      uint32_t t[32];
      tmem_ld_32x32b_x32(tS + lane_off + half * 64 + c * 32, t);
      tmem_ld_wait();
      const int d0 = r - (half * 64 + c * 32);           // distance to the first of these keys
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const int d = d0 - 2 * i;
        // a key past the chunk's end has a distance below zero for every token of the chunk
        float x0, x1;
        if (MEM) {
          const float2 g = *reinterpret_cast<const float2*>(&gates.g[half * 64 + c * 32 + 2 * i]);
          x0 = d >= 0 ? __uint_as_float(t[2 * i]) * (fast_exp2((g.x - mr) * LOG2E) * p.qscale) : 0.f;
          x1 = d >= 1 ? __uint_as_float(t[2 * i + 1]) * (fast_exp2((g.y - mr) * LOG2E) * p.qscale) : 0.f;
          wsum += x0 + x1;
        } else {
          x0 = d >= 0 ? __uint_as_float(t[2 * i]) * ret_pow(l2a, d) : 0.f;
          x1 = d >= 1 ? __uint_as_float(t[2 * i + 1]) * ret_pow(l2a, d - 1) : 0.f;
        }
        split_pair(x0, x1, ph[c * 16 + i], pl[c * 16 + i]);
      }
    }
    tc_fence_before();
    __syncthreads();                                     // everyone has read its scores
    tc_fence_after();
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      uint32_t a[16], b[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        a[i] = r < n ? ph[c * 16 + i] : 0u;
        b[i] = r < n ? pl[c * 16 + i] : 0u;
      }
      tmem_st_32x32b_x16(tS + lane_off + half * 32 + c * 16, a);
      tmem_st_32x32b_x16(tS + lane_off + 64 + half * 32 + c * 16, b);
    }
    tmem_st_wait();
  }
  mma.publish();
  if (leader) {
    const uint64_t dv = make_smem_desc_sw128(smem_u32(sV), RET_HALF, 1024);
#pragma unroll
    for (int ks = 0; ks < RET_C / 16; ++ks)
      umma_f16_ts(tO, tS + ks * 8, desc_advance(dv, ks * 2048), idesc_o, (zero && ks == 0) ? 0u : 1u);
#pragma unroll
    for (int ks = 0; ks < RET_C / 16; ++ks) umma_f16_ts(tO, tS + 64 + ks * 8, desc_advance(dv, ks * 2048), idesc_o, 1);
    umma_commit(mma.bar);
  }
  __syncwarp();
  // the gate, while the tensor core works
  float o[64];
  uint4 gv[8];
  const bool live = mine && r < n;
  const bf16_t* gp = p.gate + (row0 + r) * p.ld_in + static_cast<size_t>(h) * p.dvp + half * 64;
#pragma unroll
  for (int j = 0; j < 8; ++j)
    gv[j] = live && half * 64 + j * 8 < p.dvp ? *reinterpret_cast<const uint4*>(gp + j * 8) : make_uint4(0, 0, 0, 0);
  mma.wait();
  float ss = 0.f;
  if (mine) {
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      uint32_t t[32];
      tmem_ld_32x32b_x32(tO + lane_off + half * 64 + c * 32, t);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        o[c * 32 + i] = __uint_as_float(t[i]);
        ss = fmaf(o[c * 32 + i], o[c * 32 + i], ss);
      }
    }
  }
  xchg[half * 128 + r] = ss;
  if (MEM) swsum[half * 128 + r] = wsum;
  __syncthreads();
  const float tot = xchg[r] + xchg[128 + r];
  const float inv = MEM ? 1.f / (fmaxf(fabsf(swsum[r] + swsum[128 + r]), expf(-(gates.b[r] + gates.M[r]))) + MEMORY_EPS) : 1.f;
  if (!MEM && p.joint_ss && half == 0 && r < n) p.joint_ss[(row0 + r) * p.H + h] = tot;
  if (mine) {
    const float f = !MEM && p.joint_ss ? 1.f : (MEM ? p.oscale : 1.f) * inv / sqrtf(tot * inv * inv / p.dv + p.eps);
    uint4 ov[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const uint32_t g[4] = {gv[j].x, gv[j].y, gv[j].z, gv[j].w};
      uint32_t y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 g2 = unpack_bf16x2(g[e]);
        if (MEM || p.joint_ss) {
          const int c = half * 64 + j * 8 + 2 * e;
          const float2 w2 = c < p.dvp ? unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p.norm_w + h * p.dvp + c)) : make_float2(0.f, 0.f);
          y[e] = pack_bf16x2(o[j * 8 + 2 * e] * f * w2.x * sigmoid_fast(g2.x), o[j * 8 + 2 * e + 1] * f * w2.y * sigmoid_fast(g2.y));
          continue;
        }
        y[e] = pack_bf16x2(o[j * 8 + 2 * e] * f * silu_fast(g2.x), o[j * 8 + 2 * e + 1] * f * silu_fast(g2.y));
      }
      ov[j] = make_uint4(y[0], y[1], y[2], y[3]);
    }
    bf16_t* base = p.out + (row0 + quarter * 32) * p.ld_out + static_cast<size_t>(h) * p.dvp + half * 64;
    warp_store_rows_128B(hi + warp * 4096, ov, [&](int row) -> uint8_t* {
      if (quarter * 32 + row >= n || half * 64 + (lane & 7) * 8 >= p.dvp) return nullptr;
      return reinterpret_cast<uint8_t*>(base + static_cast<size_t>(row) * p.ld_out);
    });
  }
  mma.release(256);
}

template <bool MEM>
static int launch_ret(const RetParams& p, int nchunks, int nlong, cudaStream_t stream) {
  constexpr int CONTRIB = MEM ? MEM_CONTRIB_BYTES : RET_CONTRIB_BYTES, OUT = MEM ? MEM_OUT_BYTES : RET_OUT_BYTES;
  int* status = status_ptr();
  if (!status) return 3;
  static bool set[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!set[dev & 63]) {
    if (cudaFuncSetAttribute(ret_contrib_kernel<MEM>, cudaFuncAttributeMaxDynamicSharedMemorySize, CONTRIB) != cudaSuccess ||
        cudaFuncSetAttribute(ret_out_kernel<MEM>, cudaFuncAttributeMaxDynamicSharedMemorySize, OUT) != cudaSuccess) {
      set_error("retention_chunk: cannot set shared memory size");
      return 1;
    }
    set[dev & 63] = true;
  }
  ret_contrib_kernel<MEM><<<dim3(nchunks, p.H), RET_THREADS, CONTRIB, stream>>>(p, status);
  B2_CHECK_LAUNCH("ret_contrib");
  if (MEM) mem_scan_kernel<<<dim3(((p.dkp * p.dvp + p.dkp) / 4 + 255) / 256, p.H, nlong), 256, 0, stream>>>(p);
  else ret_scan_kernel<<<dim3((p.dkp * p.dvp / 4 + 255) / 256, p.H, nlong), 256, 0, stream>>>(p);
  B2_CHECK_LAUNCH("ret_scan");
  ret_out_kernel<MEM><<<dim3(nchunks, p.H), RET_THREADS, OUT, stream>>>(p, status);
  B2_CHECK_LAUNCH("ret_out");
  return 0;
}

}  // namespace b2

using namespace b2;

// ws: fp32 [nchunks, H, dkp, dvp].  chunks / first describe the long sequences seq0 .. seq0 + nlong - 1 in RET_C-row chunks.
B2_EXPORT int b2_retention_chunk(const void* q, const void* k, const void* v, const void* gate, void* out, float* ws,
                                 float* state, const float* decay, const float* cs, const float* sn, const int* chunks,
                                 const int* first, const int* start, const int* slot, int nchunks, int seq0, int nlong, int H,
                                 int dk, int dkp, int dv, int dvp, int rot, long long ld_in, long long ld_out, float kscale,
                                 float eps, const void* norm_w, float* joint_ss, void* stream) {
  b2::ensure_thread_context();
  if (joint_ss != nullptr && norm_w == nullptr) { set_error("retention_chunk: a joint norm needs its weight"); return 10; }
  if (nchunks <= 0 || nlong <= 0) return 0;
  if (dkp % 8 || dvp % 8 || dkp < 8 || dvp < 8 || dkp > 128 || dvp > 128 || rot < 0 || rot % 2 || rot > dk || ld_in % 8 ||
      ld_out % 8 || H < 1 || H > 65535 || nlong > 65535) {
    set_error("retention_chunk: head sizes up to 128 in multiples of 8 (padded) required");
    return 10;
  }
  RetParams p = {};
  p.q = static_cast<const bf16_t*>(q); p.k = static_cast<const bf16_t*>(k); p.v = static_cast<const bf16_t*>(v);
  p.gate = static_cast<const bf16_t*>(gate); p.out = static_cast<bf16_t*>(out); p.ws = ws; p.state = state; p.decay = decay;
  p.cs = cs; p.sn = sn; p.chunks = chunks; p.first = first; p.start = start; p.slot = slot; p.ld_in = ld_in; p.ld_out = ld_out;
  p.H = H; p.dk = dk; p.dkp = dkp; p.dv = dv; p.dvp = dvp; p.rot = rot; p.seq0 = seq0; p.kscale = kscale; p.eps = eps;
  p.norm_w = static_cast<const bf16_t*>(norm_w); p.joint_ss = joint_ss;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return launch_ret<false>(p, nchunks, nlong, st);
}

// ws as above; wn: fp32 [nchunks, H, dkp], wg: fp32 [nchunks, H, 2], wm: fp32 [nchunks, H].
B2_EXPORT int b2_memory_chunk(const void* q, const void* k, const void* v, const void* gate, const float* zi, const float* zf,
                              long long ld_z, const void* bi, const void* bf, const void* norm_w, void* out, float* ws, float* wn,
                              float* wg, float* wm, float* state, float* n, float* m, const int* chunks, const int* first,
                              const int* start, const int* slot, int nchunks, int seq0, int nlong, int H, int dk, int dkp, int dv,
                              int dvp, long long ld_in, long long ld_out, float cap, float qscale, float oscale, float eps,
                              void* stream) {
  b2::ensure_thread_context();
  if (nchunks <= 0 || nlong <= 0) return 0;
  if (dkp % 8 || dvp % 8 || dkp < 8 || dvp < 8 || dkp > 128 || dvp > 128 || ld_in % 8 || ld_out % 8 || H < 1 || H > 65535 ||
      nlong > 65535 || !(cap > 0.f)) {
    set_error("memory_chunk: head sizes up to 128 in multiples of 8 (padded) and a positive cap required");
    return 10;
  }
  RetParams p = {};
  p.q = static_cast<const bf16_t*>(q); p.k = static_cast<const bf16_t*>(k); p.v = static_cast<const bf16_t*>(v);
  p.gate = static_cast<const bf16_t*>(gate); p.out = static_cast<bf16_t*>(out); p.ws = ws; p.state = state;
  p.chunks = chunks; p.first = first; p.start = start; p.slot = slot; p.ld_in = ld_in; p.ld_out = ld_out;
  p.H = H; p.dk = dk; p.dkp = dkp; p.dv = dv; p.dvp = dvp; p.seq0 = seq0; p.kscale = 1.f; p.eps = eps;
  p.norm_w = static_cast<const bf16_t*>(norm_w);
  p.zi = zi; p.zf = zf; p.bi = static_cast<const bf16_t*>(bi); p.bf = static_cast<const bf16_t*>(bf); p.ld_z = ld_z;
  p.n = n; p.m = m; p.wn = wn; p.wg = reinterpret_cast<float2*>(wg); p.wm = wm; p.cap = cap; p.qscale = qscale; p.oscale = oscale;
  return launch_ret<true>(p, nchunks, nlong, static_cast<cudaStream_t>(stream));
}
