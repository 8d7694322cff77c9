// Paged attention one query row at a time, for any head sizes up to 256, in bf16 or true 32-bit: the decode step and short
// portions.  Beside plain causal attention it takes, each optional,
//   * chunked visibility: row at position i sees keys floor(i / chunk) * chunk .. i only;
//   * a sliding window: keys i - window + 1 .. i only;
//   * a soft cap: scores pass through cap * tanh(score / cap);
//   * a learned additive bias per head and distance bucket: rel[bucket[min(i - j, len - 1)], h];
//   * a softmax sink per head: exp(sink_h) joins the denominator, with no key and no value;
//   * an output gate per head: the head's output times sigmoid(gate);
//   * differential heads (MAPS = 2): a head has two query rows and two key rows over one value row, two attentions a1 and a2 that
//     leave as rms(a1 - lambda a2) (1 - lambda_init), times a sigmoid gate per channel.
// And the stage before it: bias, per-head RMS norm and rotary positions of q and k and the store of k and v into their pages.
//
// Cache layout of one layer: K [blocks, 16, G, dkp], V [blocks, 16, G, dvp] in the activation type, head sizes padded to a
// multiple of eight (padding zero); differential: K [blocks, 16, G, 2, dkp], q [M, H, 2, dkp].  Row r belongs to sequence row_seq[r], whose pages are block_tables[row_seq[r]][*].
#include "host.h"
#include "vec.cuh"

namespace b2 {

constexpr int AR_PAGE = 16;
constexpr int AR_THREADS = 128;
constexpr int AR_UNROLL = 4;
constexpr float AR_LOG2E = 1.4426950408889634f;

struct AttnRowsParams {
  const void* q;         // T [M, H * dkp]
  const void* kc;
  const void* vc;
  const int* tables;     // [nseq, max_blocks]
  const int* row_seq;    // [M] or null: row r is sequence r
  const int* pos;        // [M]
  const int* slot;       // per sequence, or null: slot < 0 marks a padding row (output zero)
  const void* gate;      // T [M, ld_gate]: H columns (differential: H * dvp), or null
  const void* sink;      // T [H] or null
  const void* rel;       // T [buckets, H] or null
  const int* bucket;     // [nbucket]
  void* out;             // T [M, ld_out]
  float* part_o;         // [M, H, nsplit, dvp]
  float* part_ml;        // [M, H, nsplit, 2]
  long long ld_gate, ld_out;
  int max_blocks, H, G, dkp, dvp, chunk, nbucket, partition, nsplit, groups;
  float scale;
  int window, dv;        // dv: real value channels (the differential norm divides by it)
  float softcap;
  const void* lam;       // differential: T [4, dkp] = lq1, lk1, lq2, lk2
  float lam_init, eps;
};

// softmax weights: the special-function unit's 2^x beside bf16 values, the library's in 32-bit runs
template <typename T>
__device__ __forceinline__ float ar_exp2(float x) {
  return sizeof(T) == 2 ? fast_exp2(x) : exp2f(x);
}

template <typename T>
__device__ __forceinline__ float ar_finish(const AttnRowsParams& p, int head, size_t row, float o, float L, float M2) {
  // M2: running maximum in the base-2 domain
  if (p.sink) {
    const float s2 = to_f(static_cast<const T*>(p.sink)[head]) * AR_LOG2E;
    const float m = fmaxf(M2, s2);
    const float w = M2 == -INFINITY ? 0.f : exp2f(M2 - m);
    L = L * w + exp2f(s2 - m);
    o *= w;
  }
  o = L > 0.f ? o / L : 0.f;
  if (p.gate) o *= sigmoid_f(to_f(static_cast<const T*>(p.gate)[row * p.ld_gate + head]));
  return o;
}

// Differential heads: o = a1 - lambda a2, normed over the head's channels, times 1 - lambda_init and the gate.  N channels of
// one head per thread, c0 + i * stride; `sum` adds over the threads that share the head.
template <typename T, int N, typename F>
__device__ __forceinline__ void ar_diff_store(const AttnRowsParams& p, float lam, int head, size_t row, const float (&a1)[N],
                                              const float (&a2)[N], int c0, int stride, F sum) {
  float o[N], ss = 0.f;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    o[i] = c0 + i * stride < p.dvp ? a1[i] - lam * a2[i] : 0.f;
    ss = fmaf(o[i], o[i], ss);
  }
  const float r = (1.f - p.lam_init) / sqrtf(sum(ss) / p.dv + p.eps);
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = c0 + i * stride;
    if (c >= p.dvp) break;
    float x = o[i] * r;
    if (p.gate) x *= sigmoid_t<T>(to_f(static_cast<const T*>(p.gate)[row * p.ld_gate + static_cast<size_t>(head) * p.dvp + c]));
    static_cast<T*>(p.out)[row * p.ld_out + static_cast<size_t>(head) * p.dvp + c] = from_f<T>(x);
  }
}

// Grid (M, G * groups, nsplit).  A key row is spread over LPT lanes, eight channels each, so one warp-wide step covers
// 32 / LPT tokens; every lane group runs its own online softmax over the tokens it sees for the GH query heads of this CTA,
// and groups and warps are merged at the end with the exact log-sum-exp rule.
//
// The bias of every key of the partition is looked up once, into shared memory.  bf16 rows travel through a ring of three
// stages per warp filled by 16-byte asynchronous copies (a lane reads back the bytes it copied: no barrier); 32-bit rows are
// loaded into registers.
constexpr int AR_STAGES = 3;
template <typename T>
__host__ __device__ constexpr int ar_ring_bytes(int maps) {
  return sizeof(T) == 2 ? (AR_THREADS / 32) * AR_STAGES * AR_UNROLL * (maps + 1) * 512 : 0;
}
// GH: query rows of a CTA (a differential head has two, of which row g reads key row g % 2)
template <typename T, int LPT, int GH, int MAPS>
__global__ void __launch_bounds__(AR_THREADS) attn_rows_kernel(const AttnRowsParams p) {
  constexpr int TPW = 32 / LPT, U = AR_UNROLL, PIECES = MAPS + 1;
  static_assert(GH % MAPS == 0, "a differential head's two query rows belong to one CTA");
  constexpr bool RING = sizeof(T) == 2;
  extern __shared__ __align__(16) uint8_t ar_dyn[];   // ring, then bias [GH][partition]
  __shared__ float sAcc[AR_THREADS / 32][GH][LPT * 8];
  __shared__ float sM[AR_THREADS / 32][GH], sL[AR_THREADS / 32][GH];
  const size_t row = blockIdx.x;
  const int kvh = blockIdx.y / p.groups, hg = blockIdx.y % p.groups, split = blockIdx.z;
  const int per = p.H / p.G;
  const int nh = min(GH, (per - hg * (GH / MAPS)) * MAPS);
  const int head0 = (kvh * per + hg * (GH / MAPS)) * MAPS;      // first query row's index among H * MAPS
  const int s = p.row_seq ? p.row_seq[row] : static_cast<int>(row);
  const bool live = p.slot == nullptr || p.slot[s] >= 0;
  const int pos = p.pos[row];
  const int first = p.chunk > 0 ? pos / p.chunk * p.chunk : p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int t_begin = first + split * p.partition;
  const int t_end = live ? min(pos + 1, t_begin + p.partition) : t_begin;
  const int* table = p.tables + static_cast<size_t>(s) * p.max_blocks;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, group = lane / LPT, sub = lane % LPT;
  const bool kin = sub * 8 < p.dkp, vin = sub * 8 < p.dvp;
  const T* kc = static_cast<const T*>(p.kc) + static_cast<size_t>(kvh) * MAPS * p.dkp + sub * 8;
  const T* vc = static_cast<const T*>(p.vc) + static_cast<size_t>(kvh) * p.dvp + sub * 8;
  const size_t kts = static_cast<size_t>(p.G) * MAPS * p.dkp, vts = static_cast<size_t>(p.G) * p.dvp;

  float qr[GH][8], acc[GH][8], m[GH], l[GH];
  const float qscale = p.softcap > 0.f ? p.scale : p.scale * AR_LOG2E;
#pragma unroll
  for (int g = 0; g < GH; ++g) {
    float t[8] = {};
    if (kin && g < nh) vload8(static_cast<const T*>(p.q) + (row * p.H * MAPS + head0 + g) * p.dkp + sub * 8, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      qr[g][e] = t[e] * qscale;
      acc[g][e] = 0.f;
    }
    m[g] = -INFINITY;
    l[g] = 0.f;
  }
  constexpr int STEP = (AR_THREADS / 32) * TPW * U;
  float* sBias = reinterpret_cast<float*>(ar_dyn + ar_ring_bytes<T>(MAPS));
  const uint32_t ring = smem_u32(ar_dyn) + (warp * AR_STAGES * U * PIECES * 32 + lane) * 16;
  auto issue = [&](int stage, int at) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int tok = at + u * TPW + group;
      if (tok < t_end) {
        const size_t a = static_cast<size_t>(table[tok / AR_PAGE]) * AR_PAGE + tok % AR_PAGE;
        const uint32_t dst = ring + ((stage * U + u) * PIECES) * 512;
#pragma unroll
        for (int mp = 0; mp < MAPS; ++mp)
          if (kin) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + mp * 512), "l"(kc + a * kts + mp * p.dkp) : "memory");
        if (vin) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + MAPS * 512), "l"(vc + a * vts) : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");   // one group per stage, empty ones included
  };
  int base = t_begin + warp * (TPW * U);
  if (RING) {
#pragma unroll
    for (int st = 0; st < AR_STAGES - 1; ++st) issue(st, base + st * STEP);
  }
  if (p.rel) {
    for (int i = threadIdx.x; i < t_end - t_begin; i += AR_THREADS) {
      const T* rel = static_cast<const T*>(p.rel) + static_cast<size_t>(p.bucket[min(pos - t_begin - i, p.nbucket - 1)]) * p.H + head0;
#pragma unroll
      for (int g = 0; g < GH; ++g)
        if (g < nh) sBias[g * p.partition + i] = to_f(rel[g]) * AR_LOG2E;
    }
    __syncthreads();
  }
  int stage = 0;
  for (; base < t_end; base += STEP) {
    float sc[U][GH];
    if (RING) {
      issue(stage == 0 ? AR_STAGES - 1 : stage - 1, base + (AR_STAGES - 1) * STEP);
      asm volatile("cp.async.wait_group %0;" ::"n"(AR_STAGES - 1) : "memory");
    }
    // one K (which < MAPS) or V (MAPS) piece of this lane; zero past the partition and past the head's channels
    auto piece = [&](int u, int which, float (&f)[8]) {
      const int tok = base + u * TPW + group;
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = 0.f;
      if (tok >= t_end || !(which == MAPS ? vin : kin)) return;
      if (RING) {
        vload8(reinterpret_cast<const __nv_bfloat16*>(ar_dyn + (warp * AR_STAGES * U * PIECES * 32 + lane) * 16 +
                                                      ((stage * U + u) * PIECES + which) * 512), f);
      } else {
        const size_t at = static_cast<size_t>(table[tok / AR_PAGE]) * AR_PAGE + tok % AR_PAGE;
        vload8(which == MAPS ? vc + at * vts : kc + at * kts + which * p.dkp, f);
      }
    };
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int tok = base + u * TPW + group;
      float kf[MAPS][8];
#pragma unroll
      for (int mp = 0; mp < MAPS; ++mp) piece(u, mp, kf[mp]);
#pragma unroll
      for (int g = 0; g < GH; ++g) {
        float d = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) d = fmaf(qr[g][e], kf[g % MAPS][e], d);
#pragma unroll
        for (int o = LPT / 2; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
        if (p.softcap > 0.f) d = softcap_t<T>(d, p.softcap) * AR_LOG2E;
        if (p.rel && tok < t_end && g < nh) d += sBias[g * p.partition + tok - t_begin];
        sc[u][g] = tok < t_end ? d : -INFINITY;
      }
    }
#pragma unroll
    for (int g = 0; g < GH; ++g) {
      float mn = m[g];
#pragma unroll
      for (int u = 0; u < U; ++u) mn = fmaxf(mn, sc[u][g]);
      if (mn == -INFINITY) {   // this lane group has not seen a token yet: its weights are zero
#pragma unroll
        for (int u = 0; u < U; ++u) sc[u][g] = 0.f;
        continue;
      }
      const float alpha = ar_exp2<T>(m[g] - mn);
      m[g] = mn;
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[g][e] *= alpha;
      float ps = 0.f;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        sc[u][g] = ar_exp2<T>(sc[u][g] - mn);
        ps += sc[u][g];
      }
      l[g] = l[g] * alpha + ps;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float vf[8];
      piece(u, MAPS, vf);
#pragma unroll
      for (int g = 0; g < GH; ++g)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[g][e] = fmaf(sc[u][g], vf[e], acc[g][e]);
    }
    stage = stage + 1 == AR_STAGES ? 0 : stage + 1;
  }
#pragma unroll
  for (int o = LPT; o < 32; o <<= 1)
#pragma unroll
    for (int g = 0; g < GH; ++g) {
      const float mo = __shfl_xor_sync(0xffffffffu, m[g], o), lo = __shfl_xor_sync(0xffffffffu, l[g], o);
      const float mn = fmaxf(m[g], mo);
      const float wa = m[g] == -INFINITY ? 0.f : exp2f(m[g] - mn), wb = mo == -INFINITY ? 0.f : exp2f(mo - mn);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[g][e] = acc[g][e] * wa + __shfl_xor_sync(0xffffffffu, acc[g][e], o) * wb;
      l[g] = l[g] * wa + lo * wb;
      m[g] = mn;
    }
  if (group == 0)
#pragma unroll
    for (int g = 0; g < GH; ++g) {
#pragma unroll
      for (int e = 0; e < 8; ++e) sAcc[warp][g][sub * 8 + e] = acc[g][e];
      if (sub == 0) {
        sM[warp][g] = m[g];
        sL[warp][g] = l[g];
      }
    }
  __syncthreads();
  if (MAPS == 2 && p.nsplit == 1) {
    const float lam = diff_lambda(static_cast<const T*>(p.lam), p.dkp, p.lam_init);
    for (int hd = warp; hd < nh / 2; hd += AR_THREADS / 32) {
      constexpr int N = LPT / 4;             // channels of a lane: LPT * 8 / 32
      float a[2][N];
#pragma unroll
      for (int mp = 0; mp < 2; ++mp) {
        const int g = hd * 2 + mp;
        float M = -INFINITY, L = 0.f;
#pragma unroll
        for (int w = 0; w < AR_THREADS / 32; ++w) M = fmaxf(M, sM[w][g]);
#pragma unroll
        for (int i = 0; i < N; ++i) a[mp][i] = 0.f;
#pragma unroll
        for (int w = 0; w < AR_THREADS / 32; ++w) {
          const float wt = sM[w][g] == -INFINITY ? 0.f : exp2f(sM[w][g] - M);
          L += sL[w][g] * wt;
#pragma unroll
          for (int i = 0; i < N; ++i) a[mp][i] += sAcc[w][g][lane + 32 * i] * wt;
        }
#pragma unroll
        for (int i = 0; i < N; ++i) a[mp][i] = L > 0.f ? a[mp][i] / L : 0.f;
      }
      ar_diff_store<T>(p, lam, head0 / 2 + hd, row, a[0], a[1], lane, 32, [](float v) { return warp_sum(v); });
    }
    return;
  }
  for (int i = threadIdx.x; i < nh * p.dvp; i += AR_THREADS) {
    const int g = i / p.dvp, c = i % p.dvp, head = head0 + g;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < AR_THREADS / 32; ++w) M = fmaxf(M, sM[w][g]);
    float L = 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < AR_THREADS / 32; ++w) {
      const float wt = sM[w][g] == -INFINITY ? 0.f : exp2f(sM[w][g] - M);
      L += sL[w][g] * wt;
      o += sAcc[w][g][c] * wt;
    }
    if (p.nsplit == 1) {
      static_cast<T*>(p.out)[row * p.ld_out + static_cast<size_t>(head) * p.dvp + c] = from_f<T>(ar_finish<T>(p, head, row, o, L, M));
    } else {
      const size_t at = (row * p.H * MAPS + head) * p.nsplit + split;
      p.part_o[at * p.dvp + c] = o;
      if (c == 0) {
        p.part_ml[at * 2] = M;
        p.part_ml[at * 2 + 1] = L;
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128) attn_rows_merge_kernel(const AttnRowsParams p) {
  const size_t row = blockIdx.x;
  const int head = blockIdx.y;
  const size_t at = (row * p.H + head) * p.nsplit;
  float M = -INFINITY;
  for (int i = 0; i < p.nsplit; ++i) M = fmaxf(M, p.part_ml[(at + i) * 2]);
  for (int c = threadIdx.x; c < p.dvp; c += blockDim.x) {
    float L = 0.f, o = 0.f;
    for (int i = 0; i < p.nsplit; ++i) {
      const float mi = p.part_ml[(at + i) * 2];
      if (mi == -INFINITY) continue;
      const float w = exp2f(mi - M);
      L += p.part_ml[(at + i) * 2 + 1] * w;
      o += p.part_o[(at + i) * p.dvp + c] * w;
    }
    static_cast<T*>(p.out)[row * p.ld_out + static_cast<size_t>(head) * p.dvp + c] = from_f<T>(ar_finish<T>(p, head, row, o, L, M));
  }
}

// Splits of both query rows of a differential head.  Grid (M, H).
template <typename T>
__global__ void __launch_bounds__(128) attn_rows_diff_merge_kernel(const AttnRowsParams p) {
  __shared__ float red[4];
  const size_t row = blockIdx.x;
  const int head = blockIdx.y;
  const float lam = diff_lambda(static_cast<const T*>(p.lam), p.dkp, p.lam_init);
  float a[2][2];
#pragma unroll
  for (int mp = 0; mp < 2; ++mp) {
    const size_t at = ((row * p.H + head) * 2 + mp) * p.nsplit;
    float M = -INFINITY, L = 0.f, o0 = 0.f, o1 = 0.f;
    for (int i = 0; i < p.nsplit; ++i) M = fmaxf(M, p.part_ml[(at + i) * 2]);
    for (int i = 0; i < p.nsplit; ++i) {
      const float mi = p.part_ml[(at + i) * 2];
      if (mi == -INFINITY) continue;
      const float w = exp2f(mi - M);
      L += p.part_ml[(at + i) * 2 + 1] * w;
      const float* o = p.part_o + (at + i) * p.dvp;
      if (static_cast<int>(threadIdx.x) < p.dvp) o0 += o[threadIdx.x] * w;
      if (static_cast<int>(threadIdx.x) + 128 < p.dvp) o1 += o[threadIdx.x + 128] * w;
    }
    a[mp][0] = L > 0.f ? o0 / L : 0.f;
    a[mp][1] = L > 0.f ? o1 / L : 0.f;
  }
  ar_diff_store<T>(p, lam, head, row, a[0], a[1], threadIdx.x, 128, [&](float v) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    return red[0] + red[1] + red[2] + red[3];
  });
}

struct NormStoreParams {
  const void* q;      // T rows of stride ld: H heads; k: G heads, v: Gv heads likewise
  const void* k;
  const void* v;
  void* q_out;        // T [M, H * dkp]
  void* kc;
  void* vc;
  const int* tables;
  const int* row_seq;
  const int* pos;
  const int* slot;
  const void* wq;     // T [dkp] or null
  const void* wk;
  const void* bq;     // T, the columns of q, k, v, or null
  const void* bk;
  const void* bv;
  const float* cs;    // [M, rot / 2] or null
  const float* sn;
  long long ld;
  int M, max_blocks, H, G, Gv, dk, dkp, dvp, norm, rot;
  float eps;
};

// Bias, per-head RMS norm of q and k (optional weights), rotary positions on channel pairs (2 i, 2 i + 1), and the store of k / v.
// Grid (M, y).  LPH lanes per head, eight channels each; a lane takes NS_UNROLL heads of its row at a time, their loads together.
// What waits in registers waits packed, so that eight CTAs fit on an SM.
template <typename T, int LPH, int NS_UNROLL>
__global__ void __launch_bounds__(128, sizeof(T) == 2 ? 8 : 4) qk_norm_store_kernel(const NormStoreParams p) {
  constexpr int GROUPS = 128 / LPH;
  const int group = threadIdx.x / LPH, c = threadIdx.x % LPH * 8, units = p.H + p.G + p.Gv;
  const int stride = GROUPS * gridDim.y;
  const bool kin = c < p.dkp, vin = c < p.dvp;
  Packed8<T> wq, wk;
  wq.zero();
  wk.zero();
  if (p.wq && kin) wq.load(static_cast<const T*>(p.wq) + c);
  if (p.wk && kin) wk.load(static_cast<const T*>(p.wk) + c);
  for (size_t row = blockIdx.x; row < static_cast<size_t>(p.M); row += gridDim.x) {
    const int s = p.row_seq ? p.row_seq[row] : static_cast<int>(row), pos = p.pos[row];
    const bool live = p.slot == nullptr || p.slot[s] >= 0;
    const size_t at = live ? static_cast<size_t>(p.tables[static_cast<size_t>(s) * p.max_blocks + pos / AR_PAGE]) * AR_PAGE + pos % AR_PAGE : 0;
    float co[4], si[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      co[e] = 1.f;
      si[e] = 0.f;
    }
    if (p.cs && c < p.rot) {
      const size_t f = row * (p.rot / 2) + c / 2;
      if (p.rot % 8 == 0) {
        const float4 a = *reinterpret_cast<const float4*>(p.cs + f), b = *reinterpret_cast<const float4*>(p.sn + f);
        co[0] = a.x; co[1] = a.y; co[2] = a.z; co[3] = a.w;
        si[0] = b.x; si[1] = b.y; si[2] = b.z; si[3] = b.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (c + 2 * e < p.rot) {
            co[e] = p.cs[f + e];
            si[e] = p.sn[f + e];
          }
      }
    }
    for (int w0 = blockIdx.y * GROUPS + group; __any_sync(0xffffffffu, w0 < units); w0 += stride * NS_UNROLL) {
      Packed8<T> raw[NS_UNROLL];
      auto part = [&](int w, const void* q, const void* k, const void* v) {      // the head's columns in a row of q | k | v
        return w < p.H ? static_cast<const T*>(q) + static_cast<size_t>(w) * p.dkp
                       : w < p.H + p.G ? static_cast<const T*>(k) + static_cast<size_t>(w - p.H) * p.dkp
                                       : static_cast<const T*>(v) + static_cast<size_t>(w - p.H - p.G) * p.dvp;
      };
#pragma unroll
      for (int i = 0; i < NS_UNROLL; ++i) {
        const int w = w0 + i * stride;
        raw[i].zero();
        if (w < units && (w < p.H + p.G ? kin : vin)) raw[i].load(part(w, p.q, p.k, p.v) + row * p.ld + c);
      }
#pragma unroll
      for (int i = 0; i < NS_UNROLL; ++i) {
        const int w = w0 + i * stride;
        float t[8];
        raw[i].get(t);
        const bool qk = w < p.H + p.G, in = w < units && (qk ? kin : vin);
        if (p.bq && in) {
          float b[8];
          vload8(part(w, p.bq, p.bk, p.bv) + c, b);
#pragma unroll
          for (int e = 0; e < 8; ++e) t[e] += b[e];
        }
        if (p.norm) {
          float ss = 0.f;
#pragma unroll
          for (int e = 0; e < 8; ++e) ss = fmaf(t[e], t[e], ss);
#pragma unroll
          for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
          const float r = rsqrtf(ss / p.dk + p.eps);
          if (qk) {
            if (w < p.H ? p.wq != nullptr : p.wk != nullptr) {
              float g[8];
              (w < p.H ? wq : wk).get(g);
#pragma unroll
              for (int e = 0; e < 8; ++e) t[e] *= g[e];
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) t[e] *= r;
          }
        }
        if (p.cs && qk) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float u = t[2 * e], x = t[2 * e + 1];
            t[2 * e] = u * co[e] - x * si[e];
            t[2 * e + 1] = x * co[e] + u * si[e];
          }
        }
        if (!in || (w >= p.H && !live)) continue;
        T* dst = w < p.H ? static_cast<T*>(p.q_out) + (row * p.H + w) * p.dkp
                         : qk ? static_cast<T*>(p.kc) + (at * p.G + w - p.H) * p.dkp
                              : static_cast<T*>(p.vc) + (at * p.Gv + w - p.H - p.G) * p.dvp;
        vstore8(dst + c, t);
      }
    }
  }
}

template <typename T, int LPT>
static int launch_rows(const AttnRowsParams& p, int M, int GH, cudaStream_t stream) {
  const dim3 grid(M, p.G * p.groups, p.nsplit);
  const int smem = ar_ring_bytes<T>(p.lam ? 2 : 1) + (p.rel ? GH * p.partition * 4 : 0);
#define B2_ROWS(GHV, MAPSV)                                                                                       \
  do {                                                                                                            \
    auto kern = attn_rows_kernel<T, LPT, GHV, MAPSV>;                                                                    \
    static int set[64] = {0};                                                                                     \
    int dev = 0;                                                                                                  \
    cudaGetDevice(&dev);                                                                                          \
    if (set[dev & 63] < smem) {                                                                                   \
      if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) {         \
        set_error("attn_rows: cannot set shared memory size (%d)", smem);                                         \
        return 1;                                                                                                 \
      }                                                                                                           \
      set[dev & 63] = smem;                                                                                       \
    }                                                                                                             \
    kern<<<grid, AR_THREADS, smem, stream>>>(p);                                                                  \
  } while (0)
  if (p.lam) {
    if (GH == 2) B2_ROWS(2, 2);
    else B2_ROWS(4, 2);
  } else {
    switch (GH) {
      case 1: B2_ROWS(1, 1); break;
      case 2: B2_ROWS(2, 1); break;
      case 3: B2_ROWS(3, 1); break;
      default: B2_ROWS(4, 1); break;
    }
  }
#undef B2_ROWS
  B2_CHECK_LAUNCH("attn_rows");
  if (p.nsplit > 1 && p.lam) {
    attn_rows_diff_merge_kernel<T><<<dim3(M, p.H), 128, 0, stream>>>(p);
    B2_CHECK_LAUNCH("attn_rows_diff_merge");
  } else if (p.nsplit > 1) {
    attn_rows_merge_kernel<T><<<dim3(M, p.H), 128, 0, stream>>>(p);
    B2_CHECK_LAUNCH("attn_rows_merge");
  }
  return 0;
}

}  // namespace b2

using namespace b2;

// lam (T [4, dkp]): differential heads, whose out is normed over dv channels with eps; the gate then has H * dvp columns.
// partition: keys per split (at most 4096 with a bias), counted from the row's first visible key; nsplit * partition must cover every row's keys.
B2_EXPORT int b2_attn_rows(const void* q, const void* kc, const void* vc, const int* tables, const int* row_seq,
                           const int* pos, const int* slot, const void* gate, long long ld_gate, const void* sink,
                           const void* rel, const int* bucket, int nbucket, void* out, long long ld_out, float* part_o,
                           float* part_ml, int M, int max_blocks, int H, int G, int dkp, int dvp, int chunk, int partition,
                           int nsplit, float scale, int window, float softcap, const void* lam, float lam_init, float eps, int dv,
                           int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (H < 1 || G < 1 || H % G || dkp % 8 || dvp % 8 || dkp > 256 || dvp > 256 || dkp < 8 || dvp < 8 || nsplit < 1 ||
      nsplit > 65535 || partition < 1 || (nsplit > 1 && (part_o == nullptr || part_ml == nullptr)) ||
      (rel != nullptr && (bucket == nullptr || nbucket < 1 || partition > 4096)) || max_blocks < 1 || H > 65535 ||
      (lam != nullptr && (rel != nullptr || sink != nullptr || dv < 1 || dv > dvp))) {
    set_error("attn_rows: H %% G == 0 and head sizes up to 256 in multiples of 8 (padded) required");
    return 10;
  }
  AttnRowsParams p = {};
  p.q = q; p.kc = kc; p.vc = vc; p.tables = tables; p.row_seq = row_seq; p.pos = pos; p.slot = slot; p.gate = gate;
  p.sink = sink; p.rel = rel; p.bucket = bucket; p.out = out; p.part_o = part_o; p.part_ml = part_ml; p.ld_gate = ld_gate;
  p.ld_out = ld_out; p.max_blocks = max_blocks; p.H = H; p.G = G; p.dkp = dkp; p.dvp = dvp; p.chunk = chunk;
  p.nbucket = nbucket; p.partition = partition; p.nsplit = nsplit; p.scale = scale;
  p.window = window; p.softcap = softcap; p.lam = lam; p.lam_init = lam_init; p.eps = eps; p.dv = dv;
  const int per = H / G, most = lam ? 2 : 4;
  p.groups = (per + most - 1) / most;
  const int GH = (per + p.groups - 1) / p.groups * (lam ? 2 : 1);
  const int w = dkp > dvp ? dkp : dvp;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  B2_DISPATCH_T(is_f32, {
    if (w <= 64) return (launch_rows<T, 8>(p, M, GH, st));
    if (w <= 128) return (launch_rows<T, 16>(p, M, GH, st));
    return (launch_rows<T, 32>(p, M, GH, st));
  });
}

// G = Gv = 0: queries alone
B2_EXPORT int b2_qk_norm_store(const void* q, const void* k, const void* v, long long ld, void* q_out, void* kc, void* vc,
                               const int* tables, const int* row_seq, const int* pos, const int* slot, int M,
                               int max_blocks, int H, int G, int Gv, int dk, int dkp, int dvp, const void* wq, const void* wk,
                               int norm, float eps, const void* bq, const void* bk, const void* bv, const float* cs,
                               const float* sn, int rot, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (dkp % 8 || dvp % 8 || dkp > 256 || dvp > 256 || ld % 8 || dk < 1 || dk > dkp || max_blocks < 1 || H < 1 || G < 0 || Gv < 0 ||
      (cs != nullptr && (rot < 2 || rot % 2 || rot > dk))) {
    set_error("qk_norm_store: head sizes up to 256 in multiples of 8 (padded) required");
    return 10;
  }
  if ((bq == nullptr) != (bk == nullptr) || (bq == nullptr) != (bv == nullptr)) { set_error("qk_norm_store: all biases or none"); return 10; }
  const NormStoreParams p = {q, k, v, q_out, kc, vc, tables, row_seq, pos, slot, wq, wk, bq, bk, bv, cs, sn, ld,
                             M, max_blocks, H, G, Gv, dk, dkp, dvp, norm, rot, eps};
  const int w = dkp > dvp ? dkp : dvp, lph = w <= 64 ? 8 : w <= 128 ? 16 : 32, groups = 128 / lph;
  int y = (H + G + Gv + groups - 1) / groups;              // a head per lane group; several when the rows fill the GPU
  const int unroll = M < 8 * num_sms() || y == 1 ? 1 : y == 2 ? 2 : 4;
  y = (y + unroll - 1) / unroll;
  const dim3 grid(M < 16 * num_sms() ? M : 16 * num_sms(), y);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define B2_NORM_STORE(L)                                                      \
  do {                                                                        \
    if (unroll == 1) qk_norm_store_kernel<T, L, 1><<<grid, 128, 0, st>>>(p);  \
    else if (unroll == 2) qk_norm_store_kernel<T, L, 2><<<grid, 128, 0, st>>>(p); \
    else qk_norm_store_kernel<T, L, 4><<<grid, 128, 0, st>>>(p);              \
  } while (0)
  B2_DISPATCH_T(is_f32, {
    if (lph == 8) B2_NORM_STORE(8);
    else if (lph == 16) B2_NORM_STORE(16);
    else B2_NORM_STORE(32);
  });
#undef B2_NORM_STORE
  B2_CHECK_LAUNCH("qk_norm_store");
  return 0;
}
