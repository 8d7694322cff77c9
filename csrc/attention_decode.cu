// Decode attention on the tensor cores: one query token per row, all the query rows that read the same keys together (the heads of
// a latent cache; both maps of a key head's differential heads).  Up to sixteen of them are the rows of m16n8k16 products: at
// one token per sequence the 128-row tcgen05 tile would be seven eighths padding, and the kernel is bound by the cache's bytes.
//
// The work is a list of key tiles, row after row, group after group, cut into equal runs: one per CTA, whatever the lengths of the
// rows (decode_plan writes the running tile count).  A CTA finishes every (row, group) that lies inside its run; what a cut
// divides is left as partial sums, two slots per CTA, for the merge kernel, which has one block per cut and head.
//
// Inside a CTA one warp copies (TMA boxes of one page by 64 channels into 128-byte-swizzled tiles, a ring of stages that runs ahead
// over the ends of rows) and eight compute.  Scores: each warp a group of eight keys, and with HALVES = 2 half of the channels.  They meet in shared memory, double-buffered: one barrier per tile.  Every
// warp then takes the softmax of the whole tile in the layout of its next operand, and multiplies 16-channel pieces of the values.
#include "host.h"
#include "mma_split.cuh"
#include "vec.cuh"

namespace b2 {

constexpr int AD_PAGE = 16, AD_WARPS = 8, AD_THREADS = (AD_WARPS + 4) * 32;
// registers a thread is launched with (three warps on each quarter of the SM), and what the copying and the computing warpgroups
// take of them: 128 x 40 + 256 x 232 <= 384 x 168
constexpr int AD_REGS = 168, AD_REGS_COPY = 40, AD_REGS_MATH = 232;
static_assert(128 * AD_REGS_COPY + AD_WARPS * 32 * AD_REGS_MATH <= AD_THREADS * AD_REGS, "register split");
constexpr float AD_LOG2E = 1.4426950408889634f;
typedef __nv_bfloat16 ad_bf16;

struct DecodeParams {
  const ad_bf16* q;      // [M, ld_q]: head h's map m at (h * maps + m) * (R / maps)
  // pages of keys [tokens, G, R] and of values [tokens, G, C] come by tensor map
  int apart;             // 0: a value is the first C channels of its key row
  const int* tables;     // [nseq, max_blocks]
  const int* row_seq;    // [M] or null: row r is sequence r
  const int* pos;        // [M]
  const int* prefix;     // [M + 1] key tiles of one group before each row
  const ad_bf16* sink;   // [H] or null
  const ad_bf16* gate;   // differential: [M, ld_gate] H * C columns, or null
  const ad_bf16* lam;    // differential: [4, R / 2]
  ad_bf16* out;          // [M, ld_out]: head h at h * C
  float* part_o;         // [grid][2][16][C]
  float* part_ml;        // [grid][2][16][2]
  long long ld_q, ld_gate, ld_out;
  int M, max_blocks, H, G, hgroups, maps, R, C, window, stages;
  int heads;             // heads of a group (the last group of a kv head may have fewer)
  int dv;                // differential: real value channels
  float scale, softcap, lam_init, eps;
};

// first key of the row's first tile: the page that holds the first visible one
__device__ __forceinline__ int ad_first(int pos, int window) { return window > 0 ? max(0, pos - window + 1) / AD_PAGE * AD_PAGE : 0; }

// prefix[r] = tiles of the rows before r.  One CTA.
__global__ void __launch_bounds__(1024) decode_plan_kernel(const int* __restrict__ pos, const int* __restrict__ row_seq,
                                                           const int* __restrict__ slot, int* __restrict__ prefix, int M, int window,
                                                           int tile) {
  __shared__ int sums[32];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int carry = 0;
  for (int r0 = 0; r0 < M; r0 += 1024) {
    const int r = r0 + threadIdx.x;
    int n = 0;
    if (r < M && (slot == nullptr || slot[row_seq ? row_seq[r] : r] >= 0)) n = (pos[r] + 1 - ad_first(pos[r], window) + tile - 1) / tile;
    int s = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int t = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += t;
    }
    if (lane == 31) sums[warp] = s;
    __syncthreads();
    int w = sums[lane];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int t = __shfl_up_sync(0xffffffffu, w, o);
      if (lane >= o) w += t;
    }
    const int before = warp == 0 ? 0 : __shfl_sync(0xffffffffu, w, warp - 1);
    if (r < M) prefix[r] = carry + before + s - n;
    carry += __shfl_sync(0xffffffffu, w, 31);
    __syncthreads();
  }
  if (threadIdx.x == 0) prefix[M] = carry;
}

// A place in the list of tiles: tile t of n of (row, group).
struct DecodeAt {
  int row, group, t, n;
};
// The row whose tiles hold place x (below the total), by a whole warp: 32 probes a round.
__device__ __forceinline__ DecodeAt ad_find(const DecodeParams& p, int groups, int x) {
  int lo = 0, hi = p.M;
  const int lane = threadIdx.x & 31;
  while (hi - lo > 1) {
    const int step = (hi - lo + 31) / 32, at = min(lo + (lane + 1) * step, hi);
    const int f = __ffs(__ballot_sync(0xffffffffu, p.prefix[at] * groups > x)) - 1;
    lo += f * step;
    hi = min(lo + step, hi);
  }
  DecodeAt a;
  a.row = lo;
  const int base = p.prefix[lo];
  a.n = p.prefix[lo + 1] - base;
  x -= base * groups;
  a.group = x / a.n;
  a.t = x - a.group * a.n;
  return a;
}
// The next (row, group); rows without tiles are passed over.
__device__ __forceinline__ void ad_next(const DecodeParams& p, int groups, DecodeAt& a) {
  a.t = 0;
  if (++a.group < groups) return;
  a.group = 0;
  int b = p.prefix[a.row + 1];
  do {
    ++a.row;
    const int e = p.prefix[a.row + 1];
    a.n = e - b;
    b = e;
  } while (a.n == 0 && a.row + 1 < p.M);
}

// Query rows: an odd number of 16-byte pieces apart, so that ldmatrix meets no bank twice; whole 32-channel steps.
__host__ __device__ constexpr int ad_pitch(int channels) { return (((channels * 2 + 63) / 64 * 64) / 16 | 1) * 16; }
struct DecodeSmem {
  int kparts, vparts, stage, pitch, q, s, bars, total;    // parts: 64-channel pieces, [tile keys x 128 bytes] each
  __host__ __device__ DecodeSmem(int R, int C, bool apart, int tile, int halves, int stages) {
    kparts = (R + 63) / 64;
    vparts = apart ? (C + 63) / 64 : 0;
    stage = (kparts + vparts) * tile * 128;
    pitch = ad_pitch(R);
    q = stages * stage;                               // 2 x [16] query rows
    s = q + 2 * 16 * pitch;                           // 2 x halves x [16][tile + 8] scores
    bars = s + 2 * halves * 16 * (tile + 8) * 4;      // barriers (256 B), then [16][8] sums
    total = bars + 256 + 16 * 8 * 4 + 1024;
  }
};
__device__ __forceinline__ void ad_consumer_barrier() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// QP: 32-channel steps of a warp's share of the keys; NG: 16-channel pieces of values per warp; EXACT: the sizes fill both, so that
// the loops over them have no conditions; FEW: at most eight query rows, so that the upper half of the sixteen is left out of the
// softmax.
template <int HALVES, int QP, int NG, bool EXACT, bool FEW>
__global__ void __launch_bounds__(AD_THREADS, 1) decode_attn_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const DecodeParams p, int* status) {
  constexpr int KT = 64 / HALVES, LDS = KT + 8, KS = KT / 16, PAGES = KT / AD_PAGE;
  extern __shared__ uint8_t ad_raw[];
  uint8_t* ad_smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ad_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const DecodeSmem L(p.R, p.C, p.apart, KT, HALVES, p.stages);
  uint64_t* full = reinterpret_cast<uint64_t*>(ad_smem + L.bars);
  uint64_t *empty = full + 8, *q_full = full + 16, *q_empty = full + 18;
  float* sums = reinterpret_cast<float*>(ad_smem + L.bars + 256);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int groups = p.G * p.hgroups, total = p.prefix[p.M] * groups;
  const int quota = (total + gridDim.x - 1) / gridDim.x, x0 = blockIdx.x * quota, x1 = min(x0 + quota, total);
  // what no copy ever writes of the query rows (a head's other map, missing heads, padding) is zero
  for (int i = L.q + tid * 16; i < L.s; i += AD_THREADS * 16) *reinterpret_cast<uint4*>(ad_smem + i) = make_uint4(0, 0, 0, 0);
  if (tid == 0) {
    for (int i = 0; i < 8; ++i) {
      mbar_init(full + i, 1);
      mbar_init(empty + i, AD_WARPS);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(q_full + i, 1);
      mbar_init(q_empty + i, AD_WARPS);
    }
    mbar_fence_init();
  }
  fence_proxy_async_smem();
  __syncthreads();
  if (x0 >= x1) return;
  DecodeAt a = ad_find(p, groups, x0);
  const int kq = p.R / p.maps;

  // A wait that runs out sets the status word; everyone runs on to the end (later waits return at once).
  if (warp >= AD_WARPS) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(AD_REGS_COPY));
    int st = 0, seg = 0;
    uint32_t ph = 0;
    const int parts = L.kparts + L.vparts;
    for (int x = warp == AD_WARPS ? x0 : x1; x < x1; ++seg) {      // one warp of the group copies
      const int t1 = min(a.n, a.t + x1 - x), kvh = a.group / p.hgroups, head0 = kvh * (p.H / p.G) + a.group % p.hgroups * p.heads;
      const int rows = min(p.heads, (kvh + 1) * (p.H / p.G) - head0) * p.maps, qs = seg & 1;
      const int pos = p.pos[a.row], first = ad_first(pos, p.window);
      const int* table = p.tables + static_cast<size_t>(p.row_seq ? p.row_seq[a.row] : a.row) * p.max_blocks;
      mbar_wait_warp(&q_empty[qs], ((seg >> 1) & 1) ^ 1, status, ERR_ATTN_WAIT);
      if (lane == 0) mbar_expect_tx(&q_full[qs], rows * kq * 2);
      __syncwarp();
      if (lane < rows)
        bulk_load(ad_smem + L.q + (qs * 16 + lane) * L.pitch + lane % p.maps * kq * 2,
                  p.q + a.row * p.ld_q + static_cast<size_t>(head0 * p.maps + lane) * kq, kq * 2, &q_full[qs]);
      // boxes (page, part): pages past the row's last repeat it, those keys are masked.  A lane always copies the same page of a
      // tile; its number is fetched one tile ahead.
      static_assert(32 % PAGES == 0, "a lane's boxes share a page");
      const int mypage = first / AD_PAGE + lane % PAGES, last = pos / AD_PAGE;
      int next = table[min(mypage + a.t * PAGES, last)];
      for (int t = a.t; t < t1; ++t) {
        const int token = next * AD_PAGE;
        next = table[min(mypage + (t + 1) * PAGES, last)];
        mbar_wait_warp(&empty[st], ph ^ 1, status, ERR_ATTN_WAIT);
        if (lane == 0) mbar_expect_tx(&full[st], parts * KT * 128);
        __syncwarp();
        uint8_t* tile = ad_smem + st * L.stage + lane % PAGES * (AD_PAGE * 128);
        for (int part = lane / PAGES; part < parts; part += 32 / PAGES) {
          uint8_t* dst = tile + part * (KT * 128);
          if (part < L.kparts) tma_load_3d(dst, &tmK, &full[st], part * 64, kvh, token);
          else tma_load_3d(dst, &tmV, &full[st], (part - L.kparts) * 64, kvh, token);
        }
        if (++st == p.stages) {
          st = 0;
          ph ^= 1;
        }
      }
      x += t1 - a.t;
      if (x < x1) ad_next(p, groups, a);
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(AD_REGS_MATH));
    const int kg = warp % (8 / HALVES), kh = warp / (8 / HALVES);       // this warp's eight keys and half of the channels
    const int steps = EXACT ? HALVES * QP : (p.R + 31) / 32, cut = HALVES == 1 ? steps : (steps + 1) / 2;   // 32-channel steps of the first half
    const int mine = kh ? steps - cut : cut, first_step = kh * cut, c0 = first_step * 32;
    const float lam = p.maps == 2 ? diff_lambda(p.lam, kq, p.lam_init) : 0.f;
    const float sl2 = p.scale * AD_LOG2E;
    const float cap_in = p.softcap > 0.f ? p.scale / p.softcap : 0.f, cap_out = p.softcap * AD_LOG2E;
    const int qld = L.pitch / 2;        // in elements
    // this lane's rows of the ldmatrix reads inside a [keys x 64 channels] piece: the warp's even and odd 32-channel steps of the keys, the
    // warp's 16-channel pieces of the values
    uint32_t koff[2], voff[NG];
#pragma unroll
    for (int i = 0; i < 2; ++i)
      koff[i] = ((first_step + i) >> 1) * (KT * 128) + (kg * 8 + (lane & 7)) * 128 + (((((first_step + i) & 1) * 4 + (lane >> 3)) ^ (lane & 7)) << 4);
#pragma unroll
    for (int g = 0; g < NG; ++g) voff[g] = (lane & 15) * 128 + (((((warp + 8 * g) * 2 + (lane >> 4)) & 7) ^ (lane & 7)) << 4);
    int st = 0, seg = 0, buf = 0;
    uint32_t ph = 0;
    for (int x = x0; x < x1; ++seg) {
      const int t1 = min(a.n, a.t + x1 - x), kvh = a.group / p.hgroups, head0 = kvh * (p.H / p.G) + a.group % p.hgroups * p.heads;
      const int rows = min(p.heads, (kvh + 1) * (p.H / p.G) - head0) * p.maps, qs = seg & 1;
      const int pos = p.pos[a.row], first = ad_first(pos, p.window), keys = pos + 1 - first;
      const int skip = p.window > 0 ? max(0, pos - p.window + 1) - first : 0;     // keys of the first tile before the window
      uint32_t q[QP][2][4];
      mbar_wait_warp(&q_full[qs], (seg >> 1) & 1, status, ERR_ATTN_WAIT);
      {
        const ad_bf16* sq = reinterpret_cast<const ad_bf16*>(ad_smem + L.q + qs * 16 * L.pitch) + c0;
#pragma unroll
        for (int i = 0; i < QP; ++i)
          if (EXACT || i < mine) {
            ldsm_a_mk(sq + i * 32, qld, lane, q[i][0]);
            ldsm_a_mk(sq + i * 32 + 16, qld, lane, q[i][1]);
          }
      }
      mbar_arrive_warp(&q_empty[qs]);
      float acc[NG][2][4], m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;   // rows lane / 4 and lane / 4 + 8
#pragma unroll
      for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[g][i >> 2][i & 3] = 0.f;
      // Scores of the tile in stage `at`, scaled to the base-2 domain.  The products of one tile run under the softmax of the one
      // before: nothing waits for them until they are written to the exchange buffer.
      auto scores = [&](int at, float (&d)[2][4]) {
        const uint8_t* tile = ad_smem + at * L.stage;
#pragma unroll
        for (int i = 0; i < 8; ++i) d[i >> 2][i & 3] = 0.f;
        constexpr int BATCH = 4;
#pragma unroll
        for (int i0 = 0; i0 < QP; i0 += BATCH) {
          uint32_t b[BATCH][4];
#pragma unroll
          for (int i = 0; i < BATCH; ++i)
            if (i0 + i < QP && (EXACT || i0 + i < mine)) ldsm_x4(reinterpret_cast<const ad_bf16*>(tile + ((i0 + i) >> 1) * (KT * 128) + koff[(i0 + i) & 1]), b[i]);
#pragma unroll
          for (int i = 0; i < BATCH; ++i)
            if (i0 + i < QP && (EXACT || i0 + i < mine)) {
              const uint32_t b0[2] = {b[i][0], b[i][1]}, b1[2] = {b[i][2], b[i][3]};
              mma_bf16(d[0], q[i0 + i][0], b0);
              mma_bf16(d[1], q[i0 + i][1], b1);
            }
        }
      };
      auto publish = [&](float (&d)[2][4], float* S) {
        float v[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = d[0][i] + d[1][i];
        if (HALVES == 1 && p.softcap > 0.f) {
          float big = 0.f;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            v[i] *= cap_in;
            big = fmaxf(big, fabsf(v[i]));
          }
          if (__any_sync(0xffffffffu, big > SOFTCAP_SERIES)) {
#pragma unroll
            for (int i = 0; i < 4; ++i) v[i] = cap_out * tanh_wide(v[i]);
          } else {
#pragma unroll
            for (int i = 0; i < 4; ++i) v[i] = cap_out * tanh_series(v[i]);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i) v[i] *= sl2;
        }
        float* o = S + (kh * 16 + (lane >> 2)) * LDS + kg * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(o) = make_float2(v[0], v[1]);
        if (!FEW) *reinterpret_cast<float2*>(o + 8 * LDS) = make_float2(v[2], v[3]);
        ad_consumer_barrier();
      };
      float* const Sbuf = reinterpret_cast<float*>(ad_smem + L.s);
      float d[2][4];
      mbar_wait_warp(&full[st], ph, status, ERR_ATTN_WAIT);
      scores(st, d);
      publish(d, Sbuf + buf * (HALVES * 16 * LDS));
      for (int t = a.t; t < t1; ++t) {
        const int cur = st;
        const float* S = Sbuf + buf * (HALVES * 16 * LDS);
        buf ^= 1;
        if (++st == p.stages) {
          st = 0;
          ph ^= 1;
        }
        if (t + 1 < t1) {
          mbar_wait_warp(&full[st], ph, status, ERR_ATTN_WAIT);
          scores(st, d);
        }
        constexpr int RH = FEW ? 1 : 2;
        float s[KS][RH][4];      // [16 keys][row, row + 8][key pairs 0, 1 and 8, 9 of this lane]
#pragma unroll
        for (int ks = 0; ks < KS; ++ks)
#pragma unroll
          for (int r = 0; r < RH; ++r)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              const float* at = S + ((lane >> 2) + 8 * r) * LDS + ks * 16 + u * 8 + (lane & 3) * 2;
              float2 v = *reinterpret_cast<const float2*>(at);
              if (HALVES == 2) {
                const float2 w = *reinterpret_cast<const float2*>(at + 16 * LDS);
                v.x += w.x;
                v.y += w.y;
              }
              s[ks][r][2 * u] = v.x;
              s[ks][r][2 * u + 1] = v.y;
            }
        const int left = keys - t * KT;
        if (left < KT) {
#pragma unroll
          for (int ks = 0; ks < KS; ++ks)
#pragma unroll
            for (int i = 0; i < 4; ++i)
              if (ks * 16 + (i >> 1) * 8 + (lane & 3) * 2 + (i & 1) >= left) s[ks][0][i] = s[ks][RH - 1][i] = -INFINITY;
        }
        if (t == 0 && skip > 0) {
#pragma unroll
          for (int ks = 0; ks < KS; ++ks)
#pragma unroll
            for (int i = 0; i < 4; ++i)
              if (ks * 16 + (i >> 1) * 8 + (lane & 3) * 2 + (i & 1) < skip) s[ks][0][i] = s[ks][RH - 1][i] = -INFINITY;
        }
        float n0 = m0, n1 = m1;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks)
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            n0 = fmaxf(n0, s[ks][0][i]);
            if (!FEW) n1 = fmaxf(n1, s[ks][RH - 1][i]);
          }
#pragma unroll
        for (int o = 1; o < 4; o <<= 1) {
          n0 = fmaxf(n0, __shfl_xor_sync(0xffffffffu, n0, o));
          if (!FEW) n1 = fmaxf(n1, __shfl_xor_sync(0xffffffffu, n1, o));
        }
        const float f0 = fast_exp2(m0 - n0), f1 = FEW ? 0.f : fast_exp2(m1 - n1);      // a tile has at least one key
        m0 = n0;
        m1 = n1;
        float p0 = 0.f, p1 = 0.f;
        uint32_t pa[KS][4];
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            s[ks][0][i] = fast_exp2(s[ks][0][i] - n0);
            p0 += s[ks][0][i];
            if (!FEW) {
              s[ks][RH - 1][i] = fast_exp2(s[ks][RH - 1][i] - n1);
              p1 += s[ks][RH - 1][i];
            }
          }
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            pa[ks][2 * u] = pack_bf16x2(s[ks][0][2 * u], s[ks][0][2 * u + 1]);
            pa[ks][2 * u + 1] = FEW ? 0u : pack_bf16x2(s[ks][RH - 1][2 * u], s[ks][RH - 1][2 * u + 1]);
          }
        }
        l0 = l0 * f0 + p0;       // this lane's keys only; added over the four lanes of a row at the end
        l1 = l1 * f1 + p1;
        const uint8_t* vt = ad_smem + cur * L.stage + (p.apart ? L.kparts * (KT * 128) : 0);
#pragma unroll
        for (int g = 0; g < NG; ++g) {
          const int c = (warp + 8 * g) * 16;
          if (!EXACT && c >= p.C) break;
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            acc[g][n][0] *= f0;
            acc[g][n][1] *= f0;
            if (!FEW) {
              acc[g][n][2] *= f1;
              acc[g][n][3] *= f1;
            }
          }
#pragma unroll
          for (int ks = 0; ks < KS; ++ks) {
            uint32_t b[4];
            ldsm_x4_t(reinterpret_cast<const ad_bf16*>(vt + (c >> 6) * (KT * 128) + ks * 2048 + voff[g]), b);
            mma_n16(acc[g][0], acc[g][1], pa[ks], b);
          }
        }
        mbar_arrive_warp(&empty[cur]);
        if (t + 1 < t1) publish(d, Sbuf + buf * (HALVES * 16 * LDS));
      }
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        l0 += __shfl_xor_sync(0xffffffffu, l0, o);
        l1 += __shfl_xor_sync(0xffffffffu, l1, o);
      }
      const bool whole = a.t == 0 && t1 == a.n;
      if (!whole) {
        const size_t slot = (static_cast<size_t>(blockIdx.x) * 2 + (a.t == 0 ? 1 : 0)) * 16;
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int r = (lane >> 2) + 8 * hh;
          if (r >= rows) continue;
#pragma unroll
          for (int g = 0; g < NG; ++g)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              const int c = (warp + 8 * g) * 16 + n * 8 + (lane & 3) * 2;
              if (c < p.C) *reinterpret_cast<float2*>(p.part_o + (slot + r) * p.C + c) = make_float2(acc[g][n][2 * hh], acc[g][n][2 * hh + 1]);
            }
          if (warp == 0 && (lane & 3) == 0) {
            p.part_ml[(slot + r) * 2] = hh ? m1 : m0;
            p.part_ml[(slot + r) * 2 + 1] = hh ? l1 : l0;
          }
        }
      } else if (p.maps == 1) {
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int r = (lane >> 2) + 8 * hh;
          if (r >= rows) continue;
          float den = hh ? l1 : l0;
          if (p.sink) den += fast_exp2(__bfloat162float(p.sink[head0 + r]) * AD_LOG2E - (hh ? m1 : m0));
          const float f = 1.f / den;
#pragma unroll
          for (int g = 0; g < NG; ++g)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              const int c = (warp + 8 * g) * 16 + n * 8 + (lane & 3) * 2;
              if (c < p.C)
                *reinterpret_cast<uint32_t*>(p.out + a.row * p.ld_out + static_cast<size_t>(head0 + r) * p.C + c) =
                    pack_bf16x2(acc[g][n][2 * hh] * f, acc[g][n][2 * hh + 1] * f);
            }
        }
      } else {
        // rows 2 h and 2 h + 1 are the maps of a head: lanes four apart
        float ss[2];
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const float inv = 1.f / (hh ? l1 : l0);
          ss[hh] = 0.f;
#pragma unroll
          for (int g = 0; g < NG; ++g)
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
              for (int e = 0; e < 2; ++e) {
                const float v = acc[g][n][2 * hh + e] * inv;
                const float o = v - lam * __shfl_xor_sync(0xffffffffu, v, 4);     // meaningful in the first map's lanes
                acc[g][n][2 * hh + e] = o;
                if ((warp + 8 * g) * 16 + n * 8 + (lane & 3) * 2 + e < p.C) ss[hh] = fmaf(o, o, ss[hh]);
              }
          ss[hh] += __shfl_xor_sync(0xffffffffu, ss[hh], 1);
          ss[hh] += __shfl_xor_sync(0xffffffffu, ss[hh], 2);
          if ((lane & 3) == 0) sums[((lane >> 2) + 8 * hh) * 8 + warp] = ss[hh];
        }
        ad_consumer_barrier();
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int r = (lane >> 2) + 8 * hh, head = head0 + r / 2;
          if (r >= rows || r % 2) continue;
          float tot = 0.f;
#pragma unroll
          for (int w = 0; w < AD_WARPS; ++w) tot += sums[r * 8 + w];
          const float f = (1.f - p.lam_init) / sqrtf(tot / p.dv + p.eps);
#pragma unroll
          for (int g = 0; g < NG; ++g)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              const int c = (warp + 8 * g) * 16 + n * 8 + (lane & 3) * 2;
              if (c >= p.C) continue;
              float2 s2 = make_float2(f, f);
              if (p.gate) {
                const float2 z = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p.gate + a.row * p.ld_gate + static_cast<size_t>(head) * p.C + c));
                s2 = make_float2(f * sigmoid_fast(z.x), f * sigmoid_fast(z.y));
              }
              *reinterpret_cast<uint32_t*>(p.out + a.row * p.ld_out + static_cast<size_t>(head) * p.C + c) =
                  pack_bf16x2(acc[g][n][2 * hh] * s2.x, acc[g][n][2 * hh + 1] * s2.y);
            }
        }
        ad_consumer_barrier();     // `sums` is free again
      }
      x += t1 - a.t;
      if (x < x1) ad_next(p, groups, a);
    }
  }
  if (*reinterpret_cast<volatile int*>(status) != 0) {    // copies in flight land before shared memory goes away
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
  }
}

// One block per cut (between run b and run b + 1) and head of a group: merges what the cut divides, if it is the first cut there.
__global__ void __launch_bounds__(128) decode_merge_kernel(const DecodeParams p, int grid, int tile) {
  __shared__ float red[4];
  const int groups = p.G * p.hgroups, total = p.prefix[p.M] * groups, quota = (total + grid - 1) / grid;
  const int b = blockIdx.x + 1, x = b * quota;
  if (x >= total) return;
  const DecodeAt a = ad_find(p, groups, x);
  const int start = x - a.t;
  if (a.t == 0 || (b - 1) * quota > start) return;      // the cut divides nothing, or an earlier cut does
  const int kvh = a.group / p.hgroups, head0 = kvh * (p.H / p.G) + a.group % p.hgroups * p.heads, head = head0 + blockIdx.y;
  if (static_cast<int>(blockIdx.y) >= p.heads || head >= (kvh + 1) * (p.H / p.G)) return;
  const int last = (start + a.n - 1) / quota;           // run that holds the last piece
  const int c4 = threadIdx.x * 4;
  float o[2][4] = {};
  for (int mp = 0; mp < p.maps; ++mp) {
    const int r = blockIdx.y * p.maps + mp;
    auto slot = [&](int c) { return (static_cast<size_t>(c) * 2 + (c == b - 1 ? 1 : 0)) * 16 + r; };
    float M = -INFINITY, den = 0.f;
    for (int c = b - 1; c <= last; ++c) M = fmaxf(M, p.part_ml[slot(c) * 2]);
    for (int c = b - 1; c <= last; ++c) {
      const float w = fast_exp2(p.part_ml[slot(c) * 2] - M);
      den += p.part_ml[slot(c) * 2 + 1] * w;
      if (c4 < p.C) {
        const float4 v = *reinterpret_cast<const float4*>(p.part_o + slot(c) * p.C + c4);
        o[mp][0] = fmaf(v.x, w, o[mp][0]);
        o[mp][1] = fmaf(v.y, w, o[mp][1]);
        o[mp][2] = fmaf(v.z, w, o[mp][2]);
        o[mp][3] = fmaf(v.w, w, o[mp][3]);
      }
    }
    if (p.sink) den += fast_exp2(__bfloat162float(p.sink[head]) * AD_LOG2E - M);
    const float f = 1.f / den;
#pragma unroll
    for (int e = 0; e < 4; ++e) o[mp][e] *= f;
  }
  if (p.maps == 2) {
    const float lam = diff_lambda(p.lam, p.R / 2, p.lam_init);
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      o[0][e] -= lam * o[1][e];
      ss = fmaf(o[0][e], o[0][e], ss);
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    const float f = (1.f - p.lam_init) / sqrtf((red[0] + red[1] + red[2] + red[3]) / p.dv + p.eps);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      o[0][e] *= f;
      if (p.gate && c4 < p.C) o[0][e] *= sigmoid_fast(__bfloat162float(p.gate[a.row * p.ld_gate + static_cast<size_t>(head) * p.C + c4 + e]));
    }
  }
  if (c4 < p.C)
    *reinterpret_cast<uint2*>(p.out + a.row * p.ld_out + static_cast<size_t>(head) * p.C + c4) =
        make_uint2(pack_bf16x2(o[0][0], o[0][1]), pack_bf16x2(o[0][2], o[0][3]));
}

template <int HALVES, int QP, int NG, bool EXACT, bool FEW>
static int launch_form(DecodeParams& p, const CUtensorMap* tk, const CUtensorMap* tv, int grid, cudaStream_t stream) {
  constexpr int KT = 64 / HALVES;
  auto kern = decode_attn_kernel<HALVES, QP, NG, EXACT, FEW>;
  int stages = 8;
  while (stages > 2 && DecodeSmem(p.R, p.C, p.apart, KT, HALVES, stages).total > 232448) --stages;
  const int smem = DecodeSmem(p.R, p.C, p.apart, KT, HALVES, stages).total;
  int* status = status_ptr();
  if (!status) return 3;
  static int set[64] = {0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (set[dev & 63] < smem) {
    if (smem > 232448 || cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) {
      set_error("decode_attention: cannot set shared memory size (%d)", smem);
      return 1;
    }
    set[dev & 63] = smem;
  }
  p.stages = stages;
  kern<<<grid, AD_THREADS, smem, stream>>>(*tk, *tv, p, status);
  B2_CHECK_LAUNCH("decode_attention");
  decode_merge_kernel<<<dim3(grid - 1, p.heads), 128, 0, stream>>>(p, grid, KT);
  B2_CHECK_LAUNCH("decode_attention_merge");
  return 0;
}
template <int HALVES, int QP, int NG, bool EXACT>
static int launch_decode(DecodeParams& p, const CUtensorMap* tk, const CUtensorMap* tv, int grid, cudaStream_t stream) {
  return p.heads * p.maps <= 8 ? launch_form<HALVES, QP, NG, EXACT, true>(p, tk, tv, grid, stream)
                               : launch_form<HALVES, QP, NG, EXACT, false>(p, tk, tv, grid, stream);
}

}  // namespace b2

using namespace b2;

// Keys of a tile of the form that R channels of key and C of value take (with the values in the key rows, or apart): 0 if none.
B2_EXPORT int b2_decode_tile(int R, int C, int values_apart) {
  if (R % 8 || C % 8 || R < 8 || C < 8) return 0;
  if (values_apart) return R <= 256 && C <= 128 ? 64 : 0;
  return R <= 576 && C <= 512 && C <= R ? 32 : 0;
}

B2_EXPORT int b2_decode_plan(const int* pos, const int* row_seq, const int* slot, int* prefix, int M, int window, int tile,
                             void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (tile < 1) { set_error("decode_plan: a positive tile required"); return 10; }
  decode_plan_kernel<<<1, 1024, 0, static_cast<cudaStream_t>(stream)>>>(pos, row_seq, slot, prefix, M, window, tile);
  B2_CHECK_LAUNCH("decode_plan");
  return 0;
}

// part_o: fp32 [number of SMs, 2, 16, C], part_ml: [number of SMs, 2, 16, 2].  lam given: differential heads (two query and key
// rows of R / 2 channels each over one value row).  A soft cap needs the values apart from the keys.
B2_EXPORT int b2_decode_attention(const void* q, const void* kc, const void* vc, const int* tables, const int* row_seq,
                                  const int* pos, const int* prefix, const void* sink, const void* gate, const void* lam, void* out,
                                  float* part_o, float* part_ml, long long ld_q, long long ld_gate, long long ld_out, int M,
                                  int num_blocks, int max_blocks, int H, int G, int R, int C, int window, int dv, float scale, float softcap,
                                  float lam_init, float eps, void* stream) {
  b2::ensure_thread_context();
  if (M <= 0) return 0;
  if (H < 1 || G < 1 || H % G || b2_decode_tile(R, C, vc != nullptr) == 0 || ld_q % 8 || ld_out % 4 || ld_gate % 2 || max_blocks < 1 ||
      (lam != nullptr && (R % 16 || vc == nullptr || dv < 1 || dv > C || sink != nullptr)) || (softcap > 0.f && vc == nullptr) ||
      (lam == nullptr && gate != nullptr)) {
    set_error("decode_attention: H %% G == 0 and row sizes in multiples of 8 within the forms of b2_decode_tile required");
    return 10;
  }
  DecodeParams p = {};
  p.q = static_cast<const ad_bf16*>(q); p.apart = vc != nullptr;
  p.tables = tables; p.row_seq = row_seq; p.pos = pos; p.prefix = prefix; p.sink = static_cast<const ad_bf16*>(sink);
  p.gate = static_cast<const ad_bf16*>(gate); p.lam = static_cast<const ad_bf16*>(lam); p.out = static_cast<ad_bf16*>(out);
  p.part_o = part_o; p.part_ml = part_ml; p.ld_q = ld_q; p.ld_gate = ld_gate; p.ld_out = ld_out; p.M = M;
  p.max_blocks = max_blocks; p.H = H; p.G = G; p.R = R; p.C = C; p.window = window; p.dv = dv; p.scale = scale;
  p.softcap = softcap; p.lam_init = lam_init; p.eps = eps; p.maps = lam ? 2 : 1;
  const int per = H / G, most = 16 / p.maps;
  p.hgroups = (per + most - 1) / most;
  p.heads = (per + p.hgroups - 1) / p.hgroups;
  p.hgroups = (per + p.heads - 1) / p.heads;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int grid = num_sms();
  auto map = [&](const void* base, uint64_t d) {
    const uint64_t dims[3] = {d, static_cast<uint64_t>(G), static_cast<uint64_t>(num_blocks) * AD_PAGE}, strides[2] = {d * 2, G * d * 2};
    const uint32_t box[3] = {64, 1, AD_PAGE};
    return tensor_map_nd_bf16(base, 3, dims, strides, box, 3);
  };
  const CUtensorMap *tk = map(kc, R), *tv = vc ? map(vc, C) : tk;
  if (!tk || !tv) return 2;
  if (vc && R == 128 && C == 128) return launch_decode<1, 4, 1, true>(p, tk, tv, grid, st);
  if (vc) return R == 256 && C == 128 ? launch_decode<1, 8, 1, true>(p, tk, tv, grid, st) : launch_decode<1, 8, 1, false>(p, tk, tv, grid, st);
  return R == 576 && C == 512 ? launch_decode<2, 9, 4, true>(p, tk, tv, grid, st) : launch_decode<2, 9, 4, false>(p, tk, tv, grid, st);
}
