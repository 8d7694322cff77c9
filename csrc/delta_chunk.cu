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
  // per chunk and head: split words W, Qs, Ks [64][DK], P [64][64]; fp32 U0 [64][dvp], end [DK]
  uint32_t* W;
  uint32_t* Qs;
  uint32_t* Ks;
  uint32_t* P;
  float* U0;
  float* end;
  float* o;              // [M, H * dvp]
  float* state;          // [slots, H, dkp, dvp]
  int H, G, dkp, dvp, seq0;
};

template <int DK>
__global__ void __launch_bounds__(DEL_THREADS, 1) delta_factor_kernel(const DeltaParams p) {
  constexpr int LD = DK + 8, SEGS = DEL_THREADS / DK, SEG = DEL_C / SEGS;
  extern __shared__ __align__(16) float sm[];
  float* sG = sm;                      // cumulative log decays
  float* sE = sG + DEL_C * LD;         // decays
  float* sK = sE + DEL_C * LD;
  float* sQ = sK + DEL_C * LD;
  float* sA = sQ + DEL_C * LD;         // [64][68], beta folded in
  float* sP = sA + DEL_C * DEL_LDA;
  float* sT = sP + DEL_C * DEL_LDA;    // [SEGS][DK] segment totals
  float* sB = sT + SEGS * DK;          // beta
  const int* ch = p.chunks + blockIdx.x * 4;
  const int h = blockIdx.y, n = ch[2], kvh = h / (p.H / p.G);
  const size_t row0 = ch[1], item = static_cast<size_t>(blockIdx.x) * p.H + h;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;

  for (int i = tid; i < DEL_C * (DK / 4); i += DEL_THREADS) {
    const int t = i / (DK / 4), c = i % (DK / 4) * 4;
    float4 kv = make_float4(0.f, 0.f, 0.f, 0.f), qv = kv;
    if (t < n && c < p.dkp) {
      const size_t at = ((row0 + t) * p.G + kvh) * p.dkp + c;
      kv = *reinterpret_cast<const float4*>(p.k + at);
      qv = *reinterpret_cast<const float4*>(p.q + at);
    }
    *reinterpret_cast<float4*>(sK + t * LD + c) = kv;
    *reinterpret_cast<float4*>(sQ + t * LD + c) = qv;
  }
  if (tid < DEL_C) sB[tid] = tid < n ? p.beta[(row0 + tid) * p.H + h] : 0.f;
  {
    const int c = tid % DK, seg = tid / DK;
    float sum = 0.f;
#pragma unroll 16
    for (int i = 0; i < SEG; ++i) {
      const int t = seg * SEG + i;
      const float x = t < n && c < p.dkp ? p.glog[((row0 + t) * p.H + h) * p.dkp + c] : 0.f;
      sum += x;
      sG[t * LD + c] = sum;
      sE[t * LD + c] = expf(x);
    }
    sT[seg * DK + c] = sum;
    __syncthreads();
    float before = 0.f;
    for (int s = 0; s < seg; ++s) before += sT[s * DK + c];
    if (seg > 0)
      for (int i = 0; i < SEG; ++i) sG[(seg * SEG + i) * LD + c] += before;
  }
  for (int i = tid; i < DEL_C * DEL_C; i += DEL_THREADS) {
    sA[i / DEL_C * DEL_LDA + i % DEL_C] = 0.f;
    sP[i / DEL_C * DEL_LDA + i % DEL_C] = 0.f;
  }
  __syncthreads();

  if (warp < 6) {   // blocks below the diagonal: (1,0) (2,0) (2,1) (3,0) (3,1) (3,2)
    const int I = warp == 0 ? 1 : warp < 3 ? 2 : 3, J = warp == 0 ? 0 : warp < 3 ? warp - 1 : warp - 3;
    float ak[2][4] = {}, aq[2][4] = {};
    const float* R = sG + (16 * I - 1) * LD;
#pragma unroll 2
    for (int ks = 0; ks < DK / 16; ++ks) {
      FragA fk, fq;
      FragB fb[2];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = 16 * I + g + (i & 1) * 8, c = ks * 16 + 2 * q4 + (i >> 1) * 8;
        const float2 G2 = *reinterpret_cast<const float2*>(sG + t * LD + c), R2 = *reinterpret_cast<const float2*>(R + c);
        const float e0 = expf(G2.x - R2.x), e1 = expf(G2.y - R2.y);
        const float2 k2 = *reinterpret_cast<const float2*>(sK + t * LD + c), q2 = *reinterpret_cast<const float2*>(sQ + t * LD + c);
        split_pair(k2.x * e0, k2.y * e1, fk.hi[i], fk.lo[i]);
        split_pair(q2.x * e0, q2.y * e1, fq.hi[i], fq.lo[i]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int t = 16 * J + j * 8 + g, c = ks * 16 + 2 * q4 + i * 8;
          const float2 G2 = *reinterpret_cast<const float2*>(sG + t * LD + c), R2 = *reinterpret_cast<const float2*>(R + c);
          const float2 k2 = *reinterpret_cast<const float2*>(sK + t * LD + c);
          split_pair(k2.x * expf(R2.x - G2.x), k2.y * expf(R2.y - G2.y), fb[j].hi[i], fb[j].lo[i]);
        }
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        mma_split(ak[j], fk, fb[j]);
        mma_split(aq[j], fq, fb[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int t = 16 * I + g + (r >> 1) * 8, c = 16 * J + j * 8 + 2 * q4 + (r & 1);
        sA[t * DEL_LDA + c] = ak[j][r] * sB[t];
        sP[t * DEL_LDA + c] = aq[j][r];
      }
  }
  {   // diagonal blocks: two warps each (halves of the channels), a lane per key j and quarter of the channels
    constexpr int NC = DK / 4;
    const int I = warp >> 1, j = lane & 15, c0 = (warp & 1) * (DK / 2) + (lane >> 4) * NC;
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
    // the two warps of a block add up: one writes, the other adds
    for (int pass = 0; pass < 2; ++pass) {
      if ((warp & 1) == pass && lane < 16)
#pragma unroll
        for (int t = 0; t < 16; ++t) {
          const int row = 16 * I + t;
          float* A = sA + row * DEL_LDA + 16 * I + j;
          float* P = sP + row * DEL_LDA + 16 * I + j;
          if (t > j) *A += dk[t] * sB[row];
          if (t >= j) *P += dq[t];
        }
      __syncthreads();
    }
  }

  // scaled q and k, P, the chunk's total decay
  for (int i = tid; i < DEL_C * DK; i += DEL_THREADS) {
    const int t = i / DK, c = i % DK;
    const float G = sG[t * LD + c], Ge = sG[(DEL_C - 1) * LD + c];
    p.Qs[item * DEL_C * DK + i] = split_word(sQ[t * LD + c] * expf(G));
    p.Ks[item * DEL_C * DK + i] = split_word(sK[t * LD + c] * expf(Ge - G));
  }
  for (int i = tid; i < DEL_C * DEL_C; i += DEL_THREADS)
    p.P[item * DEL_C * DEL_C + i] = split_word(sP[i / DEL_C * DEL_LDA + i % DEL_C]);
  for (int c = tid; c < DK; c += DEL_THREADS) p.end[item * DK + c] = expf(sG[(DEL_C - 1) * LD + c]);

  // (I + A) X = rhs by forward substitution, one column of [W | U0] per thread
  const bool is_w = tid < DK;
  const int col = is_w ? tid : tid - DK;
  if (is_w || col < p.dvp) {
    float X[DEL_C];
#pragma unroll
    for (int t = 0; t < DEL_C; ++t) {
      float x = 0.f;
      if (is_w) x = sB[t] * sK[t * LD + col] * expf(sG[t * LD + col]);
      else if (t < n) x = sB[t] * __bfloat162float(p.v[(row0 + t) * p.H * p.dvp + static_cast<size_t>(h) * p.dvp + col]);
      float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
      for (int j = 0; j < t; j += 4) {
        const float4 a = *reinterpret_cast<const float4*>(sA + t * DEL_LDA + j);   // zero on and above the diagonal
        s0 = fmaf(a.x, X[j], s0);
        if (j + 1 < t) s1 = fmaf(a.y, X[j + 1], s1);
        if (j + 2 < t) s2 = fmaf(a.z, X[j + 2], s2);
        if (j + 3 < t) s3 = fmaf(a.w, X[j + 3], s3);
      }
      X[t] = x - ((s0 + s1) + (s2 + s3));
      if (is_w) p.W[(item * DEL_C + t) * DK + col] = split_word(X[t]);
      else p.U0[(item * DEL_C + t) * p.dvp + col] = X[t];
    }
  }
}

// Grid (value slices of 32 channels, H, long sequences).  The state slice [DK x 32] lives in fp32 MMA accumulators and, as
// split words, transposed in shared memory, where the two products that read it take it from.
constexpr int DEL_SLICE = 32;

template <int DK>
__global__ void __launch_bounds__(DEL_THREADS, 1) delta_scan_kernel(const DeltaParams p) {
  constexpr int LDM = DK + 8, LDT = DK + 4, LDP = DEL_C + 8;
  constexpr int SN = DK / 32;                  // n8 tiles of the state a warp owns (16 key rows each)
  extern __shared__ __align__(16) uint32_t smw[];
  uint32_t* sW = smw;                          // [64][LDM]
  uint32_t* sQ = sW + DEL_C * LDM;             // [64][LDM]
  uint32_t* sK = sQ + DEL_C * LDM;             // [64][LDT]
  uint32_t* sP = sK + DEL_C * LDT;             // [64][LDP]
  uint32_t* sS = sP + DEL_C * LDP;             // [32][LDM]  state, transposed
  uint32_t* sU = sS + DEL_SLICE * LDM;         // [32][LDP]  U, transposed
  const int h = blockIdx.y, s = p.seq0 + blockIdx.z, n0 = blockIdx.x * DEL_SLICE;
  const int slot = p.slot[s];
  if (slot < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3;
  const int mt = warp & 3, nb = (warp >> 2) * 2;                 // token tile / first n8 tile for U and o
  const int sm_ = DK == 128 ? warp : (warp & 3), sn = DK == 128 ? 0 : (warp >> 2) * SN;   // state tile
  const int c0 = p.first[blockIdx.z], c1 = p.first[blockIdx.z + 1];
  float* st = p.state + (static_cast<size_t>(slot) * p.H + h) * p.dkp * p.dvp;

  auto copy_rows = [&](uint32_t* dst, int ld, const uint32_t* src, int width) {
    for (int i = tid; i < DEL_C * (width / 4); i += DEL_THREADS)
      cp_async16(dst + i / (width / 4) * ld + i % (width / 4) * 4, src + static_cast<size_t>(i) * 4);
  };
  auto load_wq = [&](int c) {
    const size_t at = (static_cast<size_t>(c) * p.H + h) * DEL_C * DK;
    copy_rows(sW, LDM, p.W + at, DK);
    copy_rows(sQ, LDM, p.Qs + at, DK);
  };
  auto load_kp = [&](int c) {
    const size_t item = static_cast<size_t>(c) * p.H + h;
    copy_rows(sK, LDT, p.Ks + item * DEL_C * DK, DK);
    copy_rows(sP, LDP, p.P + item * DEL_C * DEL_C, DEL_C);
  };
  load_wq(c0);
  load_kp(c0);
  cp_async_commit();

  float S[SN][4];
  const bool fresh = p.start[s] == 0;
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int i = sm_ * 16 + g + (r >> 1) * 8, c = n0 + (sn + j) * 8 + 2 * q + (r & 1);
      S[j][r] = !fresh && i < p.dkp && c < p.dvp ? st[static_cast<size_t>(i) * p.dvp + c] : 0.f;
    }
  auto put_state = [&]() {
#pragma unroll
    for (int j = 0; j < SN; ++j)
#pragma unroll
      for (int r = 0; r < 4; ++r)
        sS[((sn + j) * 8 + 2 * q + (r & 1)) * LDM + sm_ * 16 + g + (r >> 1) * 8] = split_word(S[j][r]);
  };
  put_state();

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
    cp_async_wait<0>();
    __syncthreads();
    float w[2][4] = {}, o[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      const FragA aw = lda_mk(sW + mt * 16 * LDM + ks * 16, LDM, g, q), aq = lda_mk(sQ + mt * 16 * LDM + ks * 16, LDM, g, q);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const FragB b = ldb_nk(sS + (nb + j) * 8 * LDM + ks * 16, LDM, g, q);
        mma_split(w[j], aw, b);
        mma_split(o[j], aq, b);
      }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 4; ++r)
        sU[((nb + j) * 8 + 2 * q + (r & 1)) * LDP + mt * 16 + g + (r >> 1) * 8] = split_word(u0[j][r] - w[j][r]);
    __syncthreads();                     // U is complete; W, Q and the old state have been read
    if (c + 1 < c1) load_wq(c + 1);
    cp_async_commit();
#pragma unroll
    for (int j = 0; j < SN; ++j) {
      S[j][0] *= d0;
      S[j][1] *= d0;
      S[j][2] *= d1;
      S[j][3] *= d1;
    }
#pragma unroll
    for (int ks = 0; ks < DEL_C / 16; ++ks) {
      const FragA a = lda_km(sK + ks * 16 * LDT + sm_ * 16, LDT, g, q);
#pragma unroll
      for (int j = 0; j < SN; ++j) mma_split(S[j], a, ldb_nk(sU + (sn + j) * 8 * LDP + ks * 16, LDP, g, q));
    }
    for (int ks = 0; ks <= mt; ++ks) {
      const FragA a = lda_mk(sP + mt * 16 * LDP + ks * 16, LDP, g, q);
#pragma unroll
      for (int j = 0; j < 2; ++j) mma_split(o[j], a, ldb_nk(sU + (nb + j) * 8 * LDP + ks * 16, LDP, g, q));
    }
    put_state();
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
    if (c + 1 < c1) load_kp(c + 1);
    cp_async_commit();
  }
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int i = sm_ * 16 + g + (r >> 1) * 8, c = n0 + (sn + j) * 8 + 2 * q + (r & 1);
      if (i < p.dkp && c < p.dvp) st[static_cast<size_t>(i) * p.dvp + c] = S[j][r];
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
  y.x = pack_bf16x2(x.x * r * w0.x * sigmoid_f(gt.x), x.y * r * w0.y * sigmoid_f(gt.y));
  y.y = pack_bf16x2(x.z * r * w1.x * sigmoid_f(gt.z), x.w * r * w1.y * sigmoid_f(gt.w));
  *reinterpret_cast<uint2*>(out + row * ld_out + static_cast<size_t>(h) * dvp + c) = y;
}

template <int DK>
static int launch_delta(const DeltaParams& p, int nchunks, int nlong, cudaStream_t stream) {
  const int sm1 = (4 * DEL_C * (DK + 8) + 2 * DEL_C * DEL_LDA + DEL_THREADS + DEL_C) * 4;
  const int sm2 = (2 * DEL_C * (DK + 8) + DEL_C * (DK + 4) + DEL_C * (DEL_C + 8) + DEL_SLICE * (DK + 8) + DEL_SLICE * (DEL_C + 8)) * 4;
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
  delta_factor_kernel<DK><<<dim3(nchunks, p.H), DEL_THREADS, sm1, stream>>>(p);
  B2_CHECK_LAUNCH("delta_factor");
  delta_scan_kernel<DK><<<dim3((p.dvp + DEL_SLICE - 1) / DEL_SLICE, p.H, nlong), DEL_THREADS, sm2, stream>>>(p);
  B2_CHECK_LAUNCH("delta_scan");
  return 0;
}

}  // namespace b2

using namespace b2;

// Words the chunked form needs per (chunk, head); the caller allocates nchunks * H times as many 32-bit words.
B2_EXPORT int b2_delta_chunk_words(int dkp, int dvp) {
  const int DK = dkp <= 64 ? 64 : 128;
  return 3 * DEL_C * DK + DEL_C * DEL_C + DEL_C * dvp + DK;
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
  p.W = static_cast<uint32_t*>(ws);
  p.Qs = p.W + items * DEL_C * DK;
  p.Ks = p.Qs + items * DEL_C * DK;
  p.P = p.Ks + items * DEL_C * DK;
  p.U0 = reinterpret_cast<float*>(p.P + items * DEL_C * DEL_C);
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
