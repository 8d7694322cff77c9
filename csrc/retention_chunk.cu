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

__device__ __forceinline__ float ret_pow(float l2a, int n) { return n == 0 ? 1.f : exp2f(l2a * n); }

// Rows of one head, rotated, times scale(t), as split words [RET_C][ld]; zero past `n` rows and past dkp channels.
template <int DK, typename F>
__device__ __forceinline__ void ret_load_rotated(uint32_t* dst, int ld, const bf16_t* src, size_t row0, int n, const RetParams& p,
                                                 F scale) {
  const int half = p.rot / 2, tid = threadIdx.x;
  if (half % 8 == 0) {
    const int rv = half / 8, pieces = rv + (DK - p.rot) / 8;   // rotated pairs of 8-channel pieces, then plain pieces
    for (int i = tid; i < RET_C * pieces; i += RET_THREADS) {
      const int t = i / pieces, c = i % pieces;
      const float f = t < n ? scale(t) : 0.f;
      uint32_t* d = dst + t * ld;
      if (c < rv) {
        float u[8] = {}, w[8] = {}, cs[8] = {}, sn[8] = {};
        if (t < n) {
          const bf16_t* s = src + (row0 + t) * p.ld_in + c * 8;
          vload8(s, u);
          vload8(s + half, w);
          vload8(p.cs + (row0 + t) * half + c * 8, cs);
          vload8(p.sn + (row0 + t) * half + c * 8, sn);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          d[c * 8 + e] = split_word((u[e] * cs[e] - w[e] * sn[e]) * f);
          d[half + c * 8 + e] = split_word((w[e] * cs[e] + u[e] * sn[e]) * f);
        }
      } else {
        const int at = p.rot + (c - rv) * 8;
        float u[8] = {};
        if (t < n && at < p.dkp) vload8(src + (row0 + t) * p.ld_in + at, u);
#pragma unroll
        for (int e = 0; e < 8; ++e) d[at + e] = split_word(u[e] * f);
      }
    }
    return;
  }
  for (int i = tid; i < RET_C * DK; i += RET_THREADS) {
    const int t = i / DK, c = i % DK;
    float x = 0.f;
    if (t < n && c < p.dkp) {
      const bf16_t* s = src + (row0 + t) * p.ld_in;
      x = to_f(s[c]);
      if (c < p.rot) {
        const int f = c < half ? c : c - half;
        const float o = to_f(s[c < half ? c + half : c - half]);
        x = x * p.cs[(row0 + t) * half + f] + (c < half ? -o : o) * p.sn[(row0 + t) * half + f];
      }
      x *= scale(t);
    }
    dst[t * ld + c] = split_word(x);
  }
}

template <int DV>
__device__ __forceinline__ void ret_load_v(bf16_t* dst, const bf16_t* src, size_t row0, int n, const RetParams& p) {
  constexpr int LDV = DV + 8;
  for (int i = threadIdx.x; i < RET_C * (DV / 8); i += RET_THREADS) {
    const int t = i / (DV / 8), c = i % (DV / 8) * 8;
    uint4 u = make_uint4(0, 0, 0, 0);
    if (t < n && c < p.dvp) u = *reinterpret_cast<const uint4*>(src + (row0 + t) * p.ld_in + c);
    *reinterpret_cast<uint4*>(dst + t * LDV + c) = u;
  }
}

template <int DK, int DV>
__global__ void __launch_bounds__(RET_THREADS) ret_contrib_kernel(const RetParams p) {
  constexpr int LDK = DK + 4, LDV = DV + 8;
  constexpr int NT = DV / 8 / (DK == 128 ? 1 : 2);   // n8 tiles per warp
  extern __shared__ __align__(16) uint8_t sm_raw[];
  uint32_t* sK = reinterpret_cast<uint32_t*>(sm_raw);
  bf16_t* sV = reinterpret_cast<bf16_t*>(sK + RET_C * LDK);
  const int* ch = p.chunks + blockIdx.x * 4;
  const int h = blockIdx.y, n = ch[2];
  const size_t row0 = ch[1];
  const float l2a = static_cast<float>(log2(static_cast<double>(p.decay[h])));
  ret_load_rotated<DK>(sK, LDK, p.k + static_cast<size_t>(h) * p.dkp, row0, n, p,
                       [&](int t) { return p.kscale * ret_pow(l2a, n - 1 - t); });
  ret_load_v<DV>(sV, p.v + static_cast<size_t>(h) * p.dvp, row0, n, p);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int mt = DK == 128 ? warp : (warp & 3), nb = DK == 128 ? 0 : (warp >> 2) * NT;
  float acc[NT][4] = {};
  for (int k0 = 0; k0 < n; k0 += 16) {
    const FragA a = lda_km(sK + k0 * LDK + mt * 16, LDK, g, q);
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      uint32_t b0[2], b1[2];
      ldb_kn_bf16_x2(sV + k0 * LDV + (nb + j) * 8, LDV, lane, b0, b1);
      mma_split_bx(acc[j], a, b0);
      mma_split_bx(acc[j + 1], a, b1);
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
  const double l2a = log2(static_cast<double>(p.decay[h]));
  float* st = p.state + (static_cast<size_t>(slot) * p.H + h) * size + i;
  float4 S = p.start[s] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st);
  const int c0 = p.first[blockIdx.z], c1 = p.first[blockIdx.z + 1];
  const size_t step = static_cast<size_t>(p.H) * size;
  float* w = p.ws + (static_cast<size_t>(c0) * p.H + h) * size + i;
  constexpr int U = 4;
  for (int c = c0; c < c1; c += U) {
    float4 kv[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (c + u < c1) kv[u] = *reinterpret_cast<const float4*>(w + u * step);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u >= c1) break;
      *reinterpret_cast<float4*>(w + u * step) = S;
      const float a = static_cast<float>(exp2(l2a * p.chunks[(c + u) * 4 + 2]));
      S.x = fmaf(a, S.x, kv[u].x);
      S.y = fmaf(a, S.y, kv[u].y);
      S.z = fmaf(a, S.z, kv[u].z);
      S.w = fmaf(a, S.w, kv[u].w);
    }
    w += U * step;
  }
  *reinterpret_cast<float4*>(st) = S;
}

template <int DK, int DV>
__global__ void __launch_bounds__(RET_THREADS) ret_out_kernel(const RetParams p) {
  constexpr int LDQ = DK + 8, LDS = DV + 4, LDV = DV + 8, NT = DV / 8, KS = DK / 16;
  constexpr int KB = RET_C * LDQ > DK * LDS ? RET_C * LDQ : DK * LDS;
  extern __shared__ __align__(16) uint8_t sm_raw[];
  uint32_t* sQ = reinterpret_cast<uint32_t*>(sm_raw);
  uint32_t* sK = sQ + RET_C * LDQ;                       // the state first, then the keys
  bf16_t* sV = reinterpret_cast<bf16_t*>(sK + KB);
  const int* ch = p.chunks + blockIdx.x * 4;
  const int h = blockIdx.y, s = ch[0], n = ch[2];
  const size_t row0 = ch[1];
  const bool zero = ch[3] == 0 && p.start[s] == 0;       // nothing before this chunk
  const float l2a = static_cast<float>(log2(static_cast<double>(p.decay[h])));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  ret_load_rotated<DK>(sQ, LDQ, p.q + static_cast<size_t>(h) * p.dkp, row0, n, p, [](int) { return 1.f; });
  ret_load_v<DV>(sV, p.v + static_cast<size_t>(h) * p.dvp, row0, n, p);
  float acc[NT][4] = {};
  if (!zero) {
    const float* w = p.ws + (static_cast<size_t>(blockIdx.x) * p.H + h) * p.dkp * p.dvp;
    for (int i = threadIdx.x; i < DK * (DV / 4); i += RET_THREADS) {
      const int r = i / (DV / 4), c = i % (DV / 4) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < p.dkp && c < p.dvp) x = *reinterpret_cast<const float4*>(w + static_cast<size_t>(r) * p.dvp + c);
      *reinterpret_cast<uint4*>(sK + r * LDS + c) = make_uint4(split_word(x.x), split_word(x.y), split_word(x.z), split_word(x.w));
    }
    __syncthreads();
    if (warp * 16 < n) {
#pragma unroll 2
      for (int ks = 0; ks < KS; ++ks) {
        const FragA a = lda_mk(sQ + warp * 16 * LDQ + ks * 16, LDQ, g, q);
#pragma unroll
        for (int j = 0; j < NT; ++j) mma_split(acc[j], a, ldb_kn(sK + ks * 16 * LDS + j * 8, LDS, g, q));
      }
      const float f0 = ret_pow(l2a, warp * 16 + g + 1), f1 = ret_pow(l2a, warp * 16 + g + 9);
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        acc[j][0] *= f0;
        acc[j][1] *= f0;
        acc[j][2] *= f1;
        acc[j][3] *= f1;
      }
    }
    __syncthreads();
  }
  ret_load_rotated<DK>(sK, LDQ, p.k + static_cast<size_t>(h) * p.dkp, row0, n, p, [&](int) { return p.kscale; });
  __syncthreads();
  if (warp * 16 >= n) return;
  for (int kb = 0; kb <= warp; ++kb) {          // 16 keys at a time, up to the diagonal
    float sc[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      const FragA a = lda_mk(sQ + warp * 16 * LDQ + ks * 16, LDQ, g, q);
#pragma unroll
      for (int j = 0; j < 2; ++j) mma_split(sc[j], a, ldb_nk(sK + (kb * 16 + j * 8) * LDQ + ks * 16, LDQ, g, q));
    }
    FragA pa;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int d = warp * 16 + g + 8 * r - (kb * 16 + j * 8 + 2 * q);     // distance to the first of the two keys
        const float x0 = d >= 0 ? sc[j][2 * r] * ret_pow(l2a, d) : 0.f;
        const float x1 = d >= 1 ? sc[j][2 * r + 1] * ret_pow(l2a, d - 1) : 0.f;
        split_pair(x0, x1, pa.hi[2 * j + r], pa.lo[2 * j + r]);
      }
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      uint32_t b0[2], b1[2];
      ldb_kn_bf16_x2(sV + kb * 16 * LDV + j * 8, LDV, lane, b0, b1);
      mma_split_bx(acc[j], pa, b0);
      mma_split_bx(acc[j + 1], pa, b1);
    }
  }
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
    const int t = warp * 16 + g + 8 * r;
    if (t >= n) continue;
    const bf16_t* gp = p.gate + (row0 + t) * p.ld_in + static_cast<size_t>(h) * p.dvp;
    bf16_t* op = p.out + (row0 + t) * p.ld_out + static_cast<size_t>(h) * p.dvp;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int c = j * 8 + 2 * q;
      if (c >= p.dvp) break;
      const float2 gv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(gp + c));
      const float f = r ? r1 : r0;
      *reinterpret_cast<uint32_t*>(op + c) = pack_bf16x2(acc[j][2 * r] * f * silu_f(gv.x), acc[j][2 * r + 1] * f * silu_f(gv.y));
    }
  }
}

template <int DK, int DV>
static int launch_ret(const RetParams& p, int nchunks, int nlong, cudaStream_t stream) {
  const int sm1 = RET_C * (DK + 4) * 4 + RET_C * (DV + 8) * 2;
  const int kb = RET_C * (DK + 8) > DK * (DV + 4) ? RET_C * (DK + 8) : DK * (DV + 4);
  const int sm3 = (RET_C * (DK + 8) + kb) * 4 + RET_C * (DV + 8) * 2;
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
