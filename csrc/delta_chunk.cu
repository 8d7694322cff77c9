// Gated delta rule over long prompt portions, chunk by chunk (DEL_C tokens).  With G_t the running sum of log decays inside a
// chunk (one per key channel) and S the state at its start, the token recurrence becomes
//
//   A_tj  = beta_t sum_c k_tc k_jc e^{G_tc - G_jc}  (j < t)        P_tj = sum_c q_tc k_jc e^{G_tc - G_jc}  (j <= t)
//   (I + A) W = beta (k e^G),  (I + A) U0 = beta v,   U = U0 - W S
//   o = (q e^G) S + P U,       S' = e^{G_end} S + (k e^{G_end - G})^T U
//
//   1. delta_factor: A, P, W, U0 and the scaled q and k of every chunk           (all chunks at once)
//   2. delta_scan:   U, o and S along the chunks of a sequence                   (one CTA per 32 value channels)
//   3. delta_finish: per-head norm, gate, store
//
// A decay may be arbitrarily strong, so e^{-G} is never formed.  Between different 16-token blocks the exponent is split at
// the end of the block before the row's own one, where both halves are <= 0; inside a block the decayed key is carried from
// row to row.  Products on tensor cores take fp32 operands as two bf16 numbers (mma_split.cuh).
#include "host.h"
#include "mma_split.cuh"
#include "vec.cuh"

namespace b2 {

constexpr int DEL_C = 64;
constexpr int DEL_THREADS = 256;
constexpr int DEL_LDA = 68;

struct DeltaParams {
  const float* q;        // [M, G * dkp]
  const float* k;
  const __nv_bfloat16* v;   // [M, H * dvp]
  const float* glog;     // [M, H * dkp]
  const float* beta;     // [M, H]
  const int* chunks;     // [n, 4]
  const int* first;      // [nlong + 1]
  const int* start;
  const int* slot;
  // per chunk and head one record of bf16 planes, exactly as the scan keeps them in shared memory (DelRecord); fp32
  // U0 [64][dvp], end [DK]
  __nv_bfloat16* rec;
  float* U0;
  float* end;
  float* o;              // [M, H * dvp]
  float* state;          // [slots, H, dkp, dvp]
  int H, G, dkp, dvp, seq0;
};

constexpr int FAC_THREADS = 512;

template <int DK>
struct DelFactor {
  static constexpr int LD = DK + 8, LDV = 128 + 8;
  static constexpr int G = 0;                          // [64][LD] running log2 decays
  static constexpr int E = G + DEL_C * LD;             // [64][LD] decays; later the hi and lo planes of k e^G
  static constexpr int K = E + DEL_C * LD;
  static constexpr int Q = K + DEL_C * LD;
  static constexpr int A = Q + DEL_C * LD;             // [64][68], beta folded in
  static constexpr int P = A + DEL_C * DEL_LDA;
  static constexpr int T = P + DEL_C * DEL_LDA;        // (I + A)^-1
  static constexpr int V = T + DEL_C * DEL_LDA;        // bf16 [64][LDV]
  static constexpr int Z = V + DEL_C * LDV / 2;        // [16][68]
  static constexpr int TOT = Z + 16 * DEL_LDA;         // segment totals
  static constexpr int B = TOT + FAC_THREADS;          // beta
  static constexpr int BYTES = (B + DEL_C) * 4;
};

// W and Ks hi then lo [2][64][DK + 8], P [2][64][64 + 8]; Qs hi only (q enters no recurrence).  The scan copies a record in two
// pieces, W | Qs and Ks | P.
template <int DK>
struct DelRecord {
  static constexpr int LDM = DK + 8, LDP = DEL_C + 8;
  static constexpr int W = 0, Q = W + 2 * DEL_C * LDM, K = Q + DEL_C * LDM, P = K + 2 * DEL_C * LDM;
  static constexpr int ELEMS = P + 2 * DEL_C * LDP;
};

template <int DK>
__global__ void __launch_bounds__(FAC_THREADS, 1) delta_factor_kernel(const DeltaParams p) {
  using L = DelFactor<DK>;
  using Rec = DelRecord<DK>;
  constexpr int LD = L::LD, LDV = L::LDV, SEGS = FAC_THREADS / DK, SEG = DEL_C / SEGS;
  extern __shared__ __align__(16) float sm[];
  float *sG = sm + L::G, *sE = sm + L::E, *sK = sm + L::K, *sQ = sm + L::Q, *sA = sm + L::A, *sP = sm + L::P, *sT = sm + L::T,
        *sZ = sm + L::Z, *sTot = sm + L::TOT, *sB = sm + L::B;
  __nv_bfloat16* sV = reinterpret_cast<__nv_bfloat16*>(sm + L::V);
  const int* ch = p.chunks + blockIdx.x * 4;
  const int h = blockIdx.y, n = ch[2], kvh = h / (p.H / p.G);
  const size_t row0 = ch[1], item = static_cast<size_t>(blockIdx.x) * p.H + h;
  __nv_bfloat16* rec = p.rec + item * Rec::ELEMS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;

  {
    float x[SEG];
    const int c = tid % DK, seg = tid / DK;
#pragma unroll
    for (int i = 0; i < SEG; ++i) {
      const int t = seg * SEG + i;
      // loads are unconditional, clamped to rows and channels that exist, so that they are all in flight together
      x[i] = p.glog[((row0 + min(t, n - 1)) * p.H + h) * p.dkp + min(c, p.dkp - 1)];
    }
    constexpr int NK = DEL_C * (DK / 4) / FAC_THREADS, NV = DEL_C * 16 / FAC_THREADS;
    float4 kv[NK], qv[NK];
    uint4 vv[NV];
#pragma unroll
    for (int j = 0; j < NK; ++j) {
      const int i = tid + j * FAC_THREADS, t = min(i / (DK / 4), n - 1), cc = min(i % (DK / 4) * 4, p.dkp - 4);
      const size_t at = ((row0 + t) * p.G + kvh) * p.dkp + cc;
      kv[j] = *reinterpret_cast<const float4*>(p.k + at);
      qv[j] = *reinterpret_cast<const float4*>(p.q + at);
    }
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = tid + j * FAC_THREADS, t = min(i / 16, n - 1), cc = min(i % 16 * 8, p.dvp - 8);
      vv[j] = *reinterpret_cast<const uint4*>(p.v + ((row0 + t) * p.H + h) * p.dvp + cc);
    }
#pragma unroll
    for (int i = 0; i < SEG; ++i) x[i] = seg * SEG + i < n && c < p.dkp ? x[i] * 1.4426950408889634f : 0.f;
#pragma unroll
    for (int j = 0; j < NK; ++j) {
      const int i = tid + j * FAC_THREADS, t = i / (DK / 4), cc = i % (DK / 4) * 4;
      const bool in = t < n && cc < p.dkp;
      const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
      *reinterpret_cast<float4*>(sK + t * LD + cc) = in ? kv[j] : z;
      *reinterpret_cast<float4*>(sQ + t * LD + cc) = in ? qv[j] : z;
    }
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = tid + j * FAC_THREADS, t = i / 16, cc = i % 16 * 8;
      *reinterpret_cast<uint4*>(sV + t * LDV + cc) = t < n && cc < p.dvp ? vv[j] : make_uint4(0, 0, 0, 0);
    }
    if (tid < DEL_C) sB[tid] = tid < n ? p.beta[(row0 + tid) * p.H + h] : 0.f;
    for (int i = tid; i < DEL_C * DEL_LDA / 4; i += FAC_THREADS) {
      reinterpret_cast<float4*>(sA)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      reinterpret_cast<float4*>(sP)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < SEG; ++i) {
      sE[(seg * SEG + i) * LD + c] = fast_exp2(x[i]);
      sum += x[i];
      x[i] = sum;
    }
    sTot[seg * DK + c] = sum;
    __syncthreads();
    float before = 0.f;
    for (int s = 0; s < seg; ++s) before += sTot[s * DK + c];
#pragma unroll
    for (int i = 0; i < SEG; ++i) sG[(seg * SEG + i) * LD + c] = x[i] + before;
  }
  __syncthreads();

  if (warp < 12) {   // blocks below the diagonal, (1,0) (2,0) (2,1) (3,0) (3,1) (3,2): of A by the first six warps, of P by the next
    const int b = warp % 6, I = b == 0 ? 1 : b < 3 ? 2 : 3, J = b == 0 ? 0 : b < 3 ? b - 1 : b - 3;
    const float* X = warp < 6 ? sK : sQ;
    float acc[2][4] = {};
    const float* R = sG + (16 * I - 1) * LD;
#pragma unroll 2
    for (int ks = 0; ks < DK / 16; ++ks) {
      FragA fa;
      FragB fb[2];
      float2 R2[2];
      R2[0] = *reinterpret_cast<const float2*>(R + ks * 16 + 2 * q4);
      R2[1] = *reinterpret_cast<const float2*>(R + ks * 16 + 2 * q4 + 8);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int at = (16 * I + g + (i & 1) * 8) * LD + ks * 16 + 2 * q4 + (i >> 1) * 8;
        const float2 G2 = *reinterpret_cast<const float2*>(sG + at), x2 = *reinterpret_cast<const float2*>(X + at);
        split_pair(x2.x * fast_exp2(G2.x - R2[i >> 1].x), x2.y * fast_exp2(G2.y - R2[i >> 1].y), fa.hi[i], fa.lo[i]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int at = (16 * J + j * 8 + g) * LD + ks * 16 + 2 * q4 + i * 8;
          const float2 G2 = *reinterpret_cast<const float2*>(sG + at), k2 = *reinterpret_cast<const float2*>(sK + at);
          split_pair(k2.x * fast_exp2(R2[i].x - G2.x), k2.y * fast_exp2(R2[i].y - G2.y), fb[j].hi[i], fb[j].lo[i]);
        }
      mma_split(acc[0], fa, fb[0]);
      mma_split(acc[1], fa, fb[1]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int t = 16 * I + g + (r >> 1) * 8, c = 16 * J + j * 8 + 2 * q4 + (r & 1);
        if (warp < 6) sA[t * DEL_LDA + c] = acc[j][r] * sB[t];
        else sP[t * DEL_LDA + c] = acc[j][r];
      }
  }
  {   // diagonal blocks: four warps each (quarters of the channels), a lane per key j and half of its warp's channels
    constexpr int NC = DK / 8;
    const int I = warp >> 2, j = lane & 15, c0 = (warp & 3) * (DK / 4) + (lane >> 4) * NC;
    float kd[NC];
#pragma unroll
    for (int c = 0; c < NC; ++c) kd[c] = sK[(16 * I + j) * LD + c0 + c];
    float dk[16], dq[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const int off = (16 * I + t) * LD + c0;
      float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
#pragma unroll
      for (int c = 0; c < NC; c += 4) {
        const float4 e = *reinterpret_cast<const float4*>(sE + off + c), k = *reinterpret_cast<const float4*>(sK + off + c),
                     q = *reinterpret_cast<const float4*>(sQ + off + c);
        if (t > j) {
          kd[c] *= e.x;
          kd[c + 1] *= e.y;
          kd[c + 2] *= e.z;
          kd[c + 3] *= e.w;
        }
        a0 = fmaf(k.x, kd[c], a0); a1 = fmaf(k.y, kd[c + 1], a1);
        a0 = fmaf(k.z, kd[c + 2], a0); a1 = fmaf(k.w, kd[c + 3], a1);
        b0 = fmaf(q.x, kd[c], b0); b1 = fmaf(q.y, kd[c + 1], b1);
        b0 = fmaf(q.z, kd[c + 2], b0); b1 = fmaf(q.w, kd[c + 3], b1);
      }
      dk[t] = a0 + a1;
      dq[t] = b0 + b1;
      dk[t] += __shfl_xor_sync(0xffffffffu, dk[t], 16);
      dq[t] += __shfl_xor_sync(0xffffffffu, dq[t], 16);
    }
    for (int pass = 0; pass < 4; ++pass) {      // the four warps of a block add up, one after the other
      if ((warp & 3) == pass)
#pragma unroll
        for (int t = 0; t < 16; ++t) {
          const int row = 16 * I + t, at = row * DEL_LDA + 16 * I + j;
          if (lane < 16) {
            if (t > j) sA[at] += dk[t] * sB[row];
          } else {
            if (t >= j) sP[at] += dq[t];
          }
        }
      __syncthreads();
    }
  }

  // scaled q and k, P, the chunk's total decay; k e^G into the planes where the decays were
  __nv_bfloat16* pKh = reinterpret_cast<__nv_bfloat16*>(sE);
  __nv_bfloat16* pKl = pKh + DEL_C * LD;
#pragma unroll 2
  for (int i = tid; i < DEL_C * (DK / 8); i += FAC_THREADS) {
    const int t = i / (DK / 8), c = i % (DK / 8) * 8;
    float G[8], Ge[8], k[8], q[8], kg[8];
    vload8(sG + t * LD + c, G);
    vload8(sG + (DEL_C - 1) * LD + c, Ge);
    vload8(sK + t * LD + c, k);
    vload8(sQ + t * LD + c, q);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float f = fast_exp2(G[e]);
      kg[e] = k[e] * f;
      q[e] *= f;
      k[e] *= fast_exp2(Ge[e] - G[e]);
    }
    store8_split(pKh + t * LD + c, pKl + t * LD + c, kg);
    vstore8(rec + Rec::Q + t * Rec::LDM + c, q);
    store8_split(rec + Rec::K + t * Rec::LDM + c, rec + Rec::K + (DEL_C + t) * Rec::LDM + c, k);
    if (t == DEL_C - 1) {
#pragma unroll
      for (int e = 0; e < 8; ++e) p.end[item * DK + c + e] = fast_exp2(Ge[e]);
    }
  }
  for (int i = tid; i < DEL_C * (DEL_C / 8); i += FAC_THREADS) {
    const int t = i / 8, c = i % 8 * 8;
    float x[8];
    vload8(sP + t * DEL_LDA + c, x);
    store8_split(rec + Rec::P + t * Rec::LDP + c, rec + Rec::P + (DEL_C + t) * Rec::LDP + c, x);
  }

  // T = (I + A)^-1: the diagonal blocks by substitution, then T_IJ = -T_II sum_K A_IK T_KJ block row by block row
  if (tid < DEL_C) {
    const int I = tid >> 4, c = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int j = 0; j < i; j += 2) {
        s0 = fmaf(sA[(16 * I + i) * DEL_LDA + 16 * I + j], x[j], s0);
        if (j + 1 < i) s1 = fmaf(sA[(16 * I + i) * DEL_LDA + 16 * I + j + 1], x[j + 1], s1);
      }
      x[i] = (i == c ? 1.f : 0.f) - (s0 + s1);
      sT[(16 * I + i) * DEL_LDA + 16 * I + c] = x[i];
    }
  }
  __syncthreads();
  for (int I = 1; I < 4; ++I) {
    for (int i = tid; i < I * 256; i += FAC_THREADS) {
      const int r = i / (16 * I), c = i % (16 * I);
      float z = 0.f;
#pragma unroll 4
      for (int k = c / 16 * 16; k < 16 * I; ++k) z = fmaf(sA[(16 * I + r) * DEL_LDA + k], sT[k * DEL_LDA + c], z);
      sZ[r * DEL_LDA + c] = z;
    }
    __syncthreads();
    for (int i = tid; i < I * 256; i += FAC_THREADS) {
      const int r = i / (16 * I), c = i % (16 * I);
      float z = 0.f;
#pragma unroll
      for (int k = 0; k < 16; ++k) z = fmaf(sT[(16 * I + r) * DEL_LDA + 16 * I + k], sZ[k * DEL_LDA + c], z);
      sT[(16 * I + r) * DEL_LDA + c] = -z;
    }
    __syncthreads();
  }

  // [W | U0] = (T beta) [k e^G | v]: one row tile of 16 tokens and a quarter of the columns per warp
  const int mt = warp & 3, grp = warp >> 2;
  constexpr int WN = DK / 32;                       // n8 tiles of W per warp
  float aw[WN][4] = {}, au[4][4] = {};
  for (int ks = 0; ks <= mt; ++ks) {
    uint32_t th[4], tl[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = ks * 16 + 2 * q4 + (i >> 1) * 8;
      const float2 x = *reinterpret_cast<const float2*>(sT + (mt * 16 + g + (i & 1) * 8) * DEL_LDA + c);
      split_pair(x.x * sB[c], x.y * sB[c + 1], th[i], tl[i]);
    }
#pragma unroll
    for (int j = 0; j < WN; j += 2) {
      uint32_t bh[4], bl[4];
      ldsm_b_kn(pKh + ks * 16 * LD + (grp * WN + j) * 8, LD, lane, bh);
      ldsm_b_kn(pKl + ks * 16 * LD + (grp * WN + j) * 8, LD, lane, bl);
      mma_n16(aw[j], aw[j + 1], th, bh);
      mma_n16(aw[j], aw[j + 1], th, bl);
      mma_n16(aw[j], aw[j + 1], tl, bh);
    }
#pragma unroll
    for (int j = 0; j < 4; j += 2) {
      uint32_t b[4];
      ldsm_b_kn(sV + ks * 16 * LDV + (grp * 4 + j) * 8, LDV, lane, b);
      mma_n16(au[j], au[j + 1], th, b);
      mma_n16(au[j], au[j + 1], tl, b);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = mt * 16 + g + 8 * r;
#pragma unroll
    for (int j = 0; j < WN; ++j) {
      uint32_t hi, lo;
      split_pair(aw[j][2 * r], aw[j][2 * r + 1], hi, lo);
      __nv_bfloat16* w = rec + Rec::W + t * Rec::LDM + (grp * WN + j) * 8 + 2 * q4;
      *reinterpret_cast<uint32_t*>(w) = hi;
      *reinterpret_cast<uint32_t*>(w + DEL_C * Rec::LDM) = lo;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = (grp * 4 + j) * 8 + 2 * q4;
      if (c < p.dvp)
        *reinterpret_cast<float2*>(p.U0 + (item * DEL_C + t) * p.dvp + c) = make_float2(au[j][2 * r], au[j][2 * r + 1]);
    }
  }
}

// Grid (value slices of 32 channels, H, long sequences).  The state slice [DK x 32] lives in fp32 MMA accumulators and, as
// hi and lo planes, in shared memory, where the two products that read it take it from.
constexpr int DEL_SLICE = 32;

template <int DK>
struct DelScan : DelRecord<DK> {                         // the record, then
  static constexpr int LDN = DEL_SLICE + 8;
  static constexpr int S = DelRecord<DK>::ELEMS;         // [2][DK][LDN]
  static constexpr int U = S + 2 * DK * LDN;             // [2][64][LDN]
  static constexpr int BARS = U + 2 * DEL_C * LDN;       // two mbarriers
  static constexpr int BYTES = BARS * 2 + 16;
  static constexpr int WQ_BYTES = DelRecord<DK>::K * 2, KP_BYTES = (DelRecord<DK>::ELEMS - DelRecord<DK>::K) * 2;
};

template <int DK>
__global__ void __launch_bounds__(DEL_THREADS, 1) delta_scan_kernel(const DeltaParams p, int* status) {
  using L = DelScan<DK>;
  constexpr int LDM = L::LDM, LDP = L::LDP, LDN = L::LDN;
  constexpr int SN = DK / 32;                  // n8 tiles of the state a warp owns (16 key rows each)
  extern __shared__ __align__(16) uint8_t sm_raw[];
  __nv_bfloat16* sm = reinterpret_cast<__nv_bfloat16*>(sm_raw);
  __nv_bfloat16 *sW = sm + L::W, *sQ = sm + L::Q, *sK = sm + L::K, *sP = sm + L::P, *sS = sm + L::S, *sU = sm + L::U;
  const int h = blockIdx.y, s = p.seq0 + blockIdx.z, n0 = blockIdx.x * DEL_SLICE;
  const int slot = p.slot[s];
  if (slot < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3;
  const int mt = warp & 3, nb = (warp >> 2) * 2;                 // token tile / first n8 tile for U and o
  const int sm_ = DK == 128 ? warp : (warp & 3), sn = DK == 128 ? 0 : (warp >> 2) * SN;   // state tile
  const int c0 = p.first[blockIdx.z], c1 = p.first[blockIdx.z + 1];
  float* st = p.state + (static_cast<size_t>(slot) * p.H + h) * p.dkp * p.dvp;

  uint64_t* bar = reinterpret_cast<uint64_t*>(sm + L::BARS);
  if (tid == 0) {
    mbar_init(&bar[0], 1);
    mbar_init(&bar[1], 1);
    mbar_fence_init();
  }
  __syncthreads();
  auto load = [&](int c, int which) {      // one thread: W | Qs or Ks | P of chunk c
    const __nv_bfloat16* src = p.rec + (static_cast<size_t>(c) * p.H + h) * L::ELEMS;
    const uint32_t bytes = which ? L::KP_BYTES : L::WQ_BYTES;
    mbar_expect_tx(&bar[which], bytes);
    bulk_load(sm + (which ? L::K : 0), src + (which ? L::K : 0), bytes, &bar[which]);
  };
  if (tid == 0) {
    load(c0, 0);
    load(c0, 1);
  }
  bool ok = true;

  float S[SN][4];
  const bool fresh = p.start[s] == 0;
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int i = sm_ * 16 + g + (r >> 1) * 8, c = n0 + (sn + j) * 8 + 2 * q + (r & 1);
      S[j][r] = !fresh && i < p.dkp && c < p.dvp ? st[static_cast<size_t>(i) * p.dvp + c] : 0.f;
    }
  // accumulator tile (rows m0 + g, + 8; two n8 tiles from n) into hi / lo planes [rows][LDN], `lo` elements apart
  auto put = [&](__nv_bfloat16* plane, int lo, int m0, int n, const float (&x)[4]) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      uint32_t hi, l;
      split_pair(x[2 * r], x[2 * r + 1], hi, l);
      __nv_bfloat16* d = plane + (m0 + g + 8 * r) * LDN + n + 2 * q;
      *reinterpret_cast<uint32_t*>(d) = hi;
      *reinterpret_cast<uint32_t*>(d + lo) = l;
    }
  };
#pragma unroll
  for (int j = 0; j < SN; ++j) put(sS, DK * LDN, sm_ * 16, (sn + j) * 8, S[j]);

  for (int c = c0; c < c1; ++c) {
    const size_t item = static_cast<size_t>(c) * p.H + h;
    const int row0 = p.chunks[c * 4 + 1], n = p.chunks[c * 4 + 2];
    float u0[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int cc = n0 + (nb + j) * 8 + 2 * q;
        float2 x = make_float2(0.f, 0.f);
        if (cc < p.dvp) x = *reinterpret_cast<const float2*>(p.U0 + (item * DEL_C + mt * 16 + g + 8 * r) * p.dvp + cc);
        u0[j][2 * r] = x.x;
        u0[j][2 * r + 1] = x.y;
      }
    const float d0 = p.end[item * DK + sm_ * 16 + g], d1 = p.end[item * DK + sm_ * 16 + g + 8];
    // W and Q of this chunk (K and P may still be on their way), and the state written at the end of the previous one
    ok = mbar_wait_warp(&bar[0], (c - c0) & 1, status, ERR_ATTN_WAIT) && ok;
    __syncthreads();
    float w[2][4] = {}, wl[2][4] = {}, o[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t wh[4], wlo[4], qh[4], sh[4], sl[4];
      ldsm_b_kn(sS + ks * 16 * LDN + nb * 8, LDN, lane, sh);
      ldsm_b_kn(sS + (DK + ks * 16) * LDN + nb * 8, LDN, lane, sl);
      ldsm_a_mk(sW + mt * 16 * LDM + ks * 16, LDM, lane, wh);
      ldsm_a_mk(sW + (DEL_C + mt * 16) * LDM + ks * 16, LDM, lane, wlo);
      ldsm_a_mk(sQ + mt * 16 * LDM + ks * 16, LDM, lane, qh);
      mma_n16(w[0], w[1], wh, sh);
      mma_n16(o[0], o[1], qh, sh);
      mma_n16(wl[0], wl[1], wlo, sh);
      mma_n16(o[0], o[1], qh, sl);
      mma_n16(wl[0], wl[1], wh, sl);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
#pragma unroll
      for (int r = 0; r < 4; ++r) u0[j][r] -= w[j][r] + wl[j][r];
      put(sU, DEL_C * LDN, mt * 16, (nb + j) * 8, u0[j]);
    }
    ok = mbar_wait_warp(&bar[1], (c - c0) & 1, status, ERR_ATTN_WAIT) && ok;
    __syncthreads();                     // U is complete; W, Q and the old state have been read
    if (tid == 0 && ok && c + 1 < c1) load(c + 1, 0);
#pragma unroll
    for (int j = 0; j < SN; ++j) {
      S[j][0] *= d0;
      S[j][1] *= d0;
      S[j][2] *= d1;
      S[j][3] *= d1;
    }
#pragma unroll
    for (int ks = 0; ks < DEL_C / 16; ++ks) {
      uint32_t kh[4], kl[4];
      ldsm_a_km(sK + ks * 16 * LDM + sm_ * 16, LDM, lane, kh);
      ldsm_a_km(sK + (DEL_C + ks * 16) * LDM + sm_ * 16, LDM, lane, kl);
#pragma unroll
      for (int j = 0; j < SN; j += 2) {
        uint32_t uh[4], ul[4];
        ldsm_b_kn(sU + ks * 16 * LDN + (sn + j) * 8, LDN, lane, uh);
        ldsm_b_kn(sU + (DEL_C + ks * 16) * LDN + (sn + j) * 8, LDN, lane, ul);
        mma_n16(S[j], S[j + 1], kh, uh);
        mma_n16(S[j], S[j + 1], kh, ul);
        mma_n16(S[j], S[j + 1], kl, uh);
      }
    }
#pragma unroll
    for (int j = 0; j < SN; ++j) put(sS, DK * LDN, sm_ * 16, (sn + j) * 8, S[j]);
    for (int ks = 0; ks <= mt; ++ks) {
      uint32_t ph[4], pl[4], uh[4], ul[4];
      ldsm_a_mk(sP + mt * 16 * LDP + ks * 16, LDP, lane, ph);
      ldsm_a_mk(sP + (DEL_C + mt * 16) * LDP + ks * 16, LDP, lane, pl);
      ldsm_b_kn(sU + ks * 16 * LDN + nb * 8, LDN, lane, uh);
      ldsm_b_kn(sU + (DEL_C + ks * 16) * LDN + nb * 8, LDN, lane, ul);
      mma_n16(o[0], o[1], ph, uh);
      mma_n16(o[0], o[1], ph, ul);
      mma_n16(o[0], o[1], pl, uh);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = mt * 16 + g + 8 * r, cc = n0 + (nb + j) * 8 + 2 * q;
        if (t < n && cc < p.dvp)
          *reinterpret_cast<float2*>(p.o + (static_cast<size_t>(row0 + t) * p.H + h) * p.dvp + cc) =
              make_float2(o[j][2 * r], o[j][2 * r + 1]);
      }
    __syncthreads();                     // K, P and U have been read
    if (tid == 0 && ok && c + 1 < c1) load(c + 1, 1);
  }
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int i = sm_ * 16 + g + (r >> 1) * 8, c = n0 + (sn + j) * 8 + 2 * q + (r & 1);
      if (i < p.dkp && c < p.dvp) st[static_cast<size_t>(i) * p.dvp + c] = S[j][r];
    }
  if (!ok) {   // a copy may still be on its way into shared memory
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
  }
}

// out = o / rms(o) * w * sigmoid(gate) per head: one warp per (row, head), at most 128 channels.
__global__ void __launch_bounds__(256) delta_finish_kernel(const float* __restrict__ o, const float* __restrict__ gate,
                                                           const __nv_bfloat16* __restrict__ w, __nv_bfloat16* __restrict__ out,
                                                           long long ld_gate, long long ld_out, int row0, int rows, int H, int dv,
                                                           int dvp, float eps) {
  const long long i = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (i >= static_cast<long long>(rows) * H) return;
  const size_t row = row0 + i / H;
  const int h = static_cast<int>(i % H), c = (threadIdx.x & 31) * 4;
  float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c < dvp) x = *reinterpret_cast<const float4*>(o + (row * H + h) * dvp + c);
  const float r = 1.f / sqrtf(warp_sum(x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w) / dv + eps);
  if (c >= dvp) return;
  const float4 gt = *reinterpret_cast<const float4*>(gate + row * ld_gate + static_cast<size_t>(h) * dvp + c);
  float2 w0 = make_float2(1.f, 1.f), w1 = w0;
  if (w) {
    w0 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(w + c));
    w1 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(w + c + 2));
  }
  uint2 y;
  y.x = pack_bf16x2(x.x * r * w0.x * sigmoid_fast(gt.x), x.y * r * w0.y * sigmoid_fast(gt.y));
  y.y = pack_bf16x2(x.z * r * w1.x * sigmoid_fast(gt.z), x.w * r * w1.y * sigmoid_fast(gt.w));
  *reinterpret_cast<uint2*>(out + row * ld_out + static_cast<size_t>(h) * dvp + c) = y;
}

template <int DK>
static int launch_delta(const DeltaParams& p, int nchunks, int nlong, cudaStream_t stream) {
  int* status = status_ptr();
  if (!status) return 3;
  const int sm1 = DelFactor<DK>::BYTES;
  const int sm2 = DelScan<DK>::BYTES;
  static bool set[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!set[dev & 63]) {
    if (cudaFuncSetAttribute(delta_factor_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, sm1) != cudaSuccess ||
        cudaFuncSetAttribute(delta_scan_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, sm2) != cudaSuccess) {
      set_error("delta_chunk: cannot set shared memory size");
      return 1;
    }
    set[dev & 63] = true;
  }
  delta_factor_kernel<DK><<<dim3(nchunks, p.H), FAC_THREADS, sm1, stream>>>(p);
  B2_CHECK_LAUNCH("delta_factor");
  delta_scan_kernel<DK><<<dim3((p.dvp + DEL_SLICE - 1) / DEL_SLICE, p.H, nlong), DEL_THREADS, sm2, stream>>>(p, status);
  B2_CHECK_LAUNCH("delta_scan");
  return 0;
}

}  // namespace b2

using namespace b2;

// Words the chunked form needs per (chunk, head); the caller allocates nchunks * H times as many 32-bit words.
B2_EXPORT int b2_delta_chunk_words(int dkp, int dvp) {
  return dkp <= 64 ? DelRecord<64>::ELEMS / 2 + DEL_C * dvp + 64 : DelRecord<128>::ELEMS / 2 + DEL_C * dvp + 128;
}

// rows: the rows row0 .. row0 + rows - 1 the chunks cover (for the final stage).  o: fp32 [M, H * dvp] scratch.
B2_EXPORT int b2_delta_chunk(const float* q, const float* k, const void* v, const float* glog, const float* beta,
                             const float* gate, const void* norm_w, void* out, float* state, void* ws, float* o,
                             const int* chunks, const int* first, const int* start, const int* slot, int nchunks, int seq0,
                             int nlong, int row0, int rows, int H, int G, int dk, int dkp, int dv, int dvp, long long ld_gate,
                             long long ld_out, float eps, void* stream) {
  b2::ensure_thread_context();
  if (nchunks <= 0 || nlong <= 0) return 0;
  if (dkp % 8 || dvp % 8 || dkp < 8 || dvp < 8 || dkp > 128 || dvp > 128 || G < 1 || H % G || H > 65535 || nlong > 65535 ||
      ld_gate % 4 || ld_out % 4) {
    set_error("delta_chunk: head sizes up to 128 in multiples of 8 (padded) and H %% G == 0 required");
    return 10;
  }
  const size_t items = static_cast<size_t>(nchunks) * H, DK = dkp <= 64 ? 64 : 128;
  DeltaParams p;
  p.q = q; p.k = k; p.v = static_cast<const __nv_bfloat16*>(v); p.glog = glog; p.beta = beta; p.chunks = chunks; p.first = first;
  p.start = start; p.slot = slot; p.state = state; p.o = o; p.H = H; p.G = G; p.dkp = dkp; p.dvp = dvp; p.seq0 = seq0;
  p.rec = static_cast<__nv_bfloat16*>(ws);
  p.U0 = reinterpret_cast<float*>(p.rec + items * (DK == 64 ? DelRecord<64>::ELEMS : DelRecord<128>::ELEMS));
  p.end = p.U0 + items * DEL_C * dvp;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int rc = DK == 64 ? launch_delta<64>(p, nchunks, nlong, st) : launch_delta<128>(p, nchunks, nlong, st);
  if (rc) return rc;
  const long long heads = static_cast<long long>(rows) * H;
  delta_finish_kernel<<<static_cast<int>((heads + 7) / 8), 256, 0, st>>>(o, gate, static_cast<const __nv_bfloat16*>(norm_w),
                                                                         static_cast<__nv_bfloat16*>(out), ld_gate, ld_out, row0,
                                                                         rows, H, dv, dvp, eps);
  B2_CHECK_LAUNCH("delta_finish");
  return 0;
}
