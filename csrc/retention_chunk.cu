// Retention over long prompt portions, chunk by chunk (RET_C tokens), in three launches per layer:
//
//   1. every chunk's own contribution to the state, K^T V with the decays to the chunk's end       (all chunks at once)
//   2. the running state at every chunk's start: S_c = a^n S_{c-1} + contribution                   (a scan, element-wise)
//   3. o = a^{t+1} S_c^T q + sum_{j <= t} a^{t-j} (q . k_j) v_j, per-head norm, gate, store         (all chunks at once)
//
// Products run on tensor cores with fp32 operands split into two bf16 numbers (mma_split.cuh); v is exact in bf16.
#include "host.h"
#include "mma_split.cuh"
#include "vec.cuh"

namespace b2 {

constexpr int RET_C = 128;
constexpr int RET_THREADS = 256;
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
  long long ld_in, ld_out;
  int H, dk, dkp, dv, dvp, rot, seq0;
  float kscale, eps;
};

__device__ __forceinline__ float ret_pow(float l2a, int n) { return n == 0 ? 1.f : fast_exp2(l2a * n); }

// ROWS rows of one head, rotated, times scale(t), as hi (and lo) bf16 matrices [ROWS][ld]; zero past `n` rows and dkp channels.
template <int DK, int ROWS, bool LO, typename F>
__device__ __forceinline__ void ret_load_rotated(bf16_t* hi, bf16_t* lo, int ld, const bf16_t* src, size_t row0, int n,
                                                 const RetParams& p, F scale) {
  const int half = p.rot / 2, tid = threadIdx.x, nthr = blockDim.x;
  auto put = [&](int t, int c, const float (&f)[8]) {
    if (LO) store8_split(hi + t * ld + c, lo + t * ld + c, f);
    else vstore8(hi + t * ld + c, f);
  };
  if (half % 8 == 0) {
    const int rv = half / 8, pieces = rv + (DK - p.rot) / 8;   // rotated pairs of 8-channel pieces, then plain pieces
#pragma unroll 2
    for (int i = tid; i < ROWS * pieces; i += nthr) {
      const int t = i / pieces, c = i % pieces;
      const float f = t < n ? scale(t) : 0.f;
      if (c < rv) {
        float u[8] = {}, w[8] = {}, cs[8] = {}, sn[8] = {}, x[8], y[8];
        if (t < n) {
          const bf16_t* s = src + (row0 + t) * p.ld_in + c * 8;
          vload8(s, u);
          vload8(s + half, w);
          vload8(p.cs + (row0 + t) * half + c * 8, cs);
          vload8(p.sn + (row0 + t) * half + c * 8, sn);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          x[e] = (u[e] * cs[e] - w[e] * sn[e]) * f;
          y[e] = (w[e] * cs[e] + u[e] * sn[e]) * f;
        }
        put(t, c * 8, x);
        put(t, half + c * 8, y);
      } else {
        const int at = p.rot + (c - rv) * 8;
        float u[8] = {};
        if (t < n && at < p.dkp) vload8(src + (row0 + t) * p.ld_in + at, u);
#pragma unroll
        for (int e = 0; e < 8; ++e) u[e] *= f;
        put(t, at, u);
      }
    }
    return;
  }
  for (int i = tid; i < ROWS * (DK / 8); i += nthr) {
    const int t = i / (DK / 8), c8 = i % (DK / 8) * 8;
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
    put(t, c8, x);
  }
}

template <int DV>
__device__ __forceinline__ void ret_load_v(bf16_t* dst, const bf16_t* src, size_t row0, int n, const RetParams& p) {
  constexpr int LDV = DV + 8;
#pragma unroll 4
  for (int i = threadIdx.x; i < RET_C * (DV / 8); i += blockDim.x) {
    const int t = i / (DV / 8), c = i % (DV / 8) * 8;
    uint4 u = make_uint4(0, 0, 0, 0);
    if (t < n && c < p.dvp) u = *reinterpret_cast<const uint4*>(src + (row0 + t) * p.ld_in + c);
    *reinterpret_cast<uint4*>(dst + t * LDV + c) = u;
  }
}

template <int DK, int DV>
__global__ void __launch_bounds__(RET_THREADS, 2) ret_contrib_kernel(const RetParams p) {
  constexpr int LDK = DK + 8, LDV = DV + 8;
  constexpr int NT = DV / 8 / (DK == 128 ? 1 : 2);   // n8 tiles per warp
  extern __shared__ __align__(16) uint8_t sm_raw[];
  bf16_t* sKh = reinterpret_cast<bf16_t*>(sm_raw);
  bf16_t* sKl = sKh + RET_C * LDK;
  bf16_t* sV = sKl + RET_C * LDK;
  const int* ch = p.chunks + blockIdx.x * 4;
  const int h = blockIdx.y, n = ch[2];
  const size_t row0 = ch[1];
  const float l2a = log2f(p.decay[h]);
  ret_load_rotated<DK, RET_C, true>(sKh, sKl, LDK, p.k + static_cast<size_t>(h) * p.dkp, row0, n, p,
                             [&](int t) { return p.kscale * ret_pow(l2a, n - 1 - t); });
  ret_load_v<DV>(sV, p.v + static_cast<size_t>(h) * p.dvp, row0, n, p);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int mt = DK == 128 ? warp : (warp & 3), nb = DK == 128 ? 0 : (warp >> 2) * NT;
  float acc[NT][4] = {};
  for (int k0 = 0; k0 < n; k0 += 16) {
    uint32_t ah[4], al[4];
    ldsm_a_km(sKh + k0 * LDK + mt * 16, LDK, lane, ah);
    ldsm_a_km(sKl + k0 * LDK + mt * 16, LDK, lane, al);
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      uint32_t b[4];
      ldsm_b_kn(sV + k0 * LDV + (nb + j) * 8, LDV, lane, b);
      mma_n16(acc[j], acc[j + 1], ah, b);
      mma_n16(acc[j], acc[j + 1], al, b);
    }
  }
  float* w = p.ws + (static_cast<size_t>(blockIdx.x) * p.H + h) * p.dkp * p.dvp;
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int c = (nb + j) * 8 + 2 * q;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = mt * 16 + g + 8 * r;
      if (i < p.dkp && c < p.dvp)
        *reinterpret_cast<float2*>(w + static_cast<size_t>(i) * p.dvp + c) = make_float2(acc[j][2 * r], acc[j][2 * r + 1]);
    }
  }
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
    for (int u = 0; u < U; ++u)
      if (c + u < c1) kv[u] = *reinterpret_cast<const float4*>(w + u * step);
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

// Eight warps, 16 tokens each.  The state and the keys pass through one buffer in pieces of 64 rows, so that two CTAs fit on
// an SM and one's loads run under the other's products.  Products with q take q's hi part only (q enters no recurrence).
constexpr int RET_PIECE = 64;

template <int DK, int DV>
__host__ __device__ constexpr int ret_piece_elems() {
  return 2 * RET_PIECE * (DK > DV ? DK + 8 : DV + 8);
}

template <int DK, int DV>
__global__ void __launch_bounds__(RET_THREADS, 2) ret_out_kernel(const RetParams p) {
  constexpr int LDK = DK + 8, LDV = DV + 8, NT = DV / 8, KS = DK / 16;
  extern __shared__ __align__(16) uint8_t sm_raw[];
  bf16_t* sQ = reinterpret_cast<bf16_t*>(sm_raw);
  bf16_t* sV = sQ + RET_C * LDK;
  bf16_t* hi = sV + RET_C * LDV;
  const int* ch = p.chunks + blockIdx.x * 4;
  const int h = blockIdx.y, s = ch[0], n = ch[2];
  const size_t row0 = ch[1];
  const bool zero = ch[3] == 0 && p.start[s] == 0;       // nothing before this chunk
  const float l2a = log2f(p.decay[h]);
  const int rt = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const bool active = rt * 16 < n;
  ret_load_rotated<DK, RET_C, false>(sQ, nullptr, LDK, p.q + static_cast<size_t>(h) * p.dkp, row0, n, p, [](int) { return 1.f; });
  ret_load_v<DV>(sV, p.v + static_cast<size_t>(h) * p.dvp, row0, n, p);
  float acc[NT][4] = {};
  if (!zero) {
    bf16_t* lo = hi + RET_PIECE * LDV;
    const float* w = p.ws + (static_cast<size_t>(blockIdx.x) * p.H + h) * p.dkp * p.dvp;
    for (int r0 = 0; r0 < DK; r0 += RET_PIECE) {
      if (r0 > 0) __syncthreads();
#pragma unroll 4
      for (int i = threadIdx.x; i < RET_PIECE * (DV / 8); i += RET_THREADS) {
        const int r = i / (DV / 8), c = i % (DV / 8) * 8;
        float x[8] = {};
        if (r0 + r < p.dkp && c < p.dvp) vload8(w + static_cast<size_t>(r0 + r) * p.dvp + c, x);
        store8_split(hi + r * LDV + c, lo + r * LDV + c, x);
      }
      __syncthreads();
      if (active)
#pragma unroll
        for (int ks = 0; ks < RET_PIECE / 16; ++ks) {
          uint32_t a[4];
          ldsm_a_mk(sQ + rt * 16 * LDK + r0 + ks * 16, LDK, lane, a);
#pragma unroll
          for (int j = 0; j < NT; j += 2) {
            uint32_t b[4];
            ldsm_b_kn(hi + ks * 16 * LDV + j * 8, LDV, lane, b);
            mma_n16(acc[j], acc[j + 1], a, b);
            ldsm_b_kn(lo + ks * 16 * LDV + j * 8, LDV, lane, b);
            mma_n16(acc[j], acc[j + 1], a, b);
          }
        }
    }
    const float f0 = ret_pow(l2a, rt * 16 + g + 1), f1 = ret_pow(l2a, rt * 16 + g + 9);
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      acc[j][0] *= f0;
      acc[j][1] *= f0;
      acc[j][2] *= f1;
      acc[j][3] *= f1;
    }
    __syncthreads();
  }
  bf16_t* lo = hi + RET_PIECE * LDK;
  for (int k0 = 0; k0 < n; k0 += RET_PIECE) {
    if (k0 > 0) __syncthreads();
    ret_load_rotated<DK, RET_PIECE, true>(hi, lo, LDK, p.k + static_cast<size_t>(h) * p.dkp, row0 + k0, n - k0, p,
                                          [&](int) { return p.kscale; });
    __syncthreads();
    for (int kb = 0; active && kb < RET_PIECE / 16 && k0 / 16 + kb <= rt; ++kb) {     // 16 keys at a time, up to the diagonal
      float sc[2][4] = {};
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        uint32_t a[4], b[4];
        ldsm_a_mk(sQ + rt * 16 * LDK + ks * 16, LDK, lane, a);
        ldsm_b_nk(hi + kb * 16 * LDK + ks * 16, LDK, lane, b);
        mma_n16(sc[0], sc[1], a, b);
        ldsm_b_nk(lo + kb * 16 * LDK + ks * 16, LDK, lane, b);
        mma_n16(sc[0], sc[1], a, b);
      }
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int d = rt * 16 + g + 8 * r - (k0 + kb * 16 + j * 8 + 2 * q);     // distance to the first of the two keys
          const float x0 = d >= 0 ? sc[j][2 * r] * ret_pow(l2a, d) : 0.f;
          const float x1 = d >= 1 ? sc[j][2 * r + 1] * ret_pow(l2a, d - 1) : 0.f;
          split_pair(x0, x1, ph[2 * j + r], pl[2 * j + r]);
        }
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        uint32_t b[4];
        ldsm_b_kn(sV + (k0 + kb * 16) * LDV + j * 8, LDV, lane, b);
        mma_n16(acc[j], acc[j + 1], ph, b);
        mma_n16(acc[j], acc[j + 1], pl, b);
      }
    }
  }
  if (!active) return;
  float s0 = 0.f, s1 = 0.f;
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    s0 += acc[j][0] * acc[j][0] + acc[j][1] * acc[j][1];
    s1 += acc[j][2] * acc[j][2] + acc[j][3] * acc[j][3];
  }
#pragma unroll
  for (int o = 1; o < 4; o <<= 1) {
    s0 += __shfl_xor_sync(0xffffffffu, s0, o);
    s1 += __shfl_xor_sync(0xffffffffu, s1, o);
  }
  const float r0 = 1.f / sqrtf(s0 / p.dv + p.eps), r1 = 1.f / sqrtf(s1 / p.dv + p.eps);
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = rt * 16 + g + 8 * r;
    if (t >= n) continue;
    const bf16_t* gp = p.gate + (row0 + t) * p.ld_in + static_cast<size_t>(h) * p.dvp;
    bf16_t* op = p.out + (row0 + t) * p.ld_out + static_cast<size_t>(h) * p.dvp;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int c = j * 8 + 2 * q;
      if (c >= p.dvp) break;
      const float2 gv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(gp + c));
      const float f = r ? r1 : r0;
      *reinterpret_cast<uint32_t*>(op + c) = pack_bf16x2(acc[j][2 * r] * f * silu_fast(gv.x), acc[j][2 * r + 1] * f * silu_fast(gv.y));
    }
  }
}

template <int DK, int DV>
static int launch_ret(const RetParams& p, int nchunks, int nlong, cudaStream_t stream) {
  const int sm1 = RET_C * (2 * (DK + 8) + DV + 8) * 2;
  const int sm3 = (RET_C * (DK + 8 + DV + 8) + ret_piece_elems<DK, DV>()) * 2;
  static bool set[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!set[dev & 63]) {
    if (cudaFuncSetAttribute(ret_contrib_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, sm1) != cudaSuccess ||
        cudaFuncSetAttribute(ret_out_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, sm3) != cudaSuccess) {
      set_error("retention_chunk: cannot set shared memory size");
      return 1;
    }
    set[dev & 63] = true;
  }
  ret_contrib_kernel<DK, DV><<<dim3(nchunks, p.H), RET_THREADS, sm1, stream>>>(p);
  B2_CHECK_LAUNCH("ret_contrib");
  ret_scan_kernel<<<dim3((p.dkp * p.dvp / 4 + 255) / 256, p.H, nlong), 256, 0, stream>>>(p);
  B2_CHECK_LAUNCH("ret_scan");
  ret_out_kernel<DK, DV><<<dim3(nchunks, p.H), RET_THREADS, sm3, stream>>>(p);
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
                                 float eps, void* stream) {
  b2::ensure_thread_context();
  if (nchunks <= 0 || nlong <= 0) return 0;
  if (dkp % 8 || dvp % 8 || dkp < 8 || dvp < 8 || dkp > 128 || dvp > 128 || rot < 0 || rot % 2 || rot > dk || ld_in % 8 ||
      ld_out % 8 || H < 1 || H > 65535 || nlong > 65535) {
    set_error("retention_chunk: head sizes up to 128 in multiples of 8 (padded) required");
    return 10;
  }
  RetParams p;
  p.q = static_cast<const bf16_t*>(q); p.k = static_cast<const bf16_t*>(k); p.v = static_cast<const bf16_t*>(v);
  p.gate = static_cast<const bf16_t*>(gate); p.out = static_cast<bf16_t*>(out); p.ws = ws; p.state = state; p.decay = decay;
  p.cs = cs; p.sn = sn; p.chunks = chunks; p.first = first; p.start = start; p.slot = slot; p.ld_in = ld_in; p.ld_out = ld_out;
  p.H = H; p.dk = dk; p.dkp = dkp; p.dv = dv; p.dvp = dvp; p.rot = rot; p.seq0 = seq0; p.kscale = kscale; p.eps = eps;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dkp <= 64) return dvp <= 64 ? launch_ret<64, 64>(p, nchunks, nlong, st) : launch_ret<64, 128>(p, nchunks, nlong, st);
  return dvp <= 64 ? launch_ret<128, 64>(p, nchunks, nlong, st) : launch_ret<128, 128>(p, nchunks, nlong, st);
}
