// Linear-attention recurrences with a matrix state per head, S [key channel, value channel] in fp32, kept in per-sequence
// slots and carried from token to token:
//
//   retention   S <- a_h S + k v^T                                     o = S^T q     (one fixed decay per head)
//   delta rule  S <- g . S;  u = beta (v - S^T k);  S <- S + k u^T     o = S^T q     (one decay per head and key channel)
//   memory      m <- max(f + m', i);  S <- e^{f + m' - m} S + e^{i - m} k v^T;  n likewise with k alone
//               o = S^T q / (max(|n . q|, e^{-m}) + 1e-6)              (log gates i, f per head and token; m from 0)
//
// followed by a per-head RMS norm over the value channels and an output gate; or, for retention whose heads are normed together,
// by the norm's weight and a sigmoid gate, with the sum of squares of every head left for the reader of the output projection
// (the norm is one factor per row, which commutes with that projection); memory has a norm per head with a weight for every channel
// of every head, and a sigmoid gate.  This file has the token-by-token form,
// which is the decode step, the form for short portions, and the one that runs in true 32-bit; it also has the delta
// rule's input stage (short causal convolution, activation, unit norms, decays, step sizes).
//
// A portion of a sequence is a run of rows: sequence s owns rows cu[s]..cu[s+1] of the projections, its first row sits at
// position start[s], its state in slot[s] (slot < 0: padding of a graph batch, skipped).  start == 0 means the state is
// zero, whatever the slot holds: a slot needs no clearing between two sequences.
#include "host.h"
#include "vec.cuh"

namespace b2 {

struct StateSeqs {
  const int* cu;
  const int* start;
  const int* slot;
};

struct SerialParams {
  StateSeqs seq;
  // retention: projection rows (T), row stride ld; delta: fp32 rows from the input stage
  const void* q;
  const void* k;
  const void* v;      // T in both forms
  const void* gate;   // retention: T; delta: fp32
  const float* glog;  // delta: [M, H * dkp] log decays
  const float* beta;  // delta: [M, H]
  const float* cs;    // rotary tables [M, rot / 2] (retention)
  const float* sn;
  const float* decay;       // retention: [H]
  const void* norm_w;       // T [dvp] or null; retention with joint_ss and memory: T [H * dvp]
  float* joint_ss;          // retention: [M, H], or null for a norm per head
  void* out;                // T, row stride ld_out
  float* state;             // [slots, H, dkp, dvp]
  long long ld_qk, ld_v, ld_gate, ld_out;
  int H, group;             // head h uses q / k head h / group
  int dk, dkp, dv, dvp, rot;
  float kscale, eps;
  int tile;                 // tokens staged at a time
  // memory: gates before bias and cap, fp32 [M, ld_z]; their biases T [H]; normaliser [slots, H, dkp] and running maximum [slots, H]
  const float* zi;
  const float* zf;
  const void* bi;
  const void* bf;
  float* n;
  float* m;
  long long ld_z;
  float cap, qscale, oscale;
};
enum : int { RETENTION = 0, DELTA_RULE = 1, MEMORY = 2 };
constexpr float MEMORY_EPS = 1e-6f;

// log input and log forget gate of memory
__device__ __forceinline__ float2 memory_gates(float zi, float zf, float cap) {
  const float x = cap * tanhf(zf / cap);
  return make_float2(cap * tanhf(zi / cap), fminf(x, 0.f) - log1pf(expf(-fabsf(x))));
}

// One CTA per (head, sequence).  A warp owns eight value columns; its lanes form four groups that split the key rows in
// quads (lane group r holds rows 16 j + 4 r .. + 3), so the state of a head lives in registers, 4 JJ values a thread, and
// the two reductions of a token are two shuffles.  q, k and the decays of a tile of tokens are staged in shared memory as
// fp32 (rotated / exponentiated there once); the outputs of the tile are collected in shared memory, normed, gated, stored.
template <typename T, int JJ, int KIND, int MAXT>
__global__ void __launch_bounds__(MAXT) state_serial_kernel(const SerialParams p) {
  constexpr int DK = 16 * JJ;
  constexpr bool DELTA = KIND == DELTA_RULE, MEM = KIND == MEMORY;
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.x, s = blockIdx.y;
  const int slot = p.seq.slot[s];
  const int row0 = p.seq.cu[s], count = p.seq.cu[s + 1] - row0;
  if (slot < 0 || count <= 0) return;
  const int TT = p.tile;
  float* sk = sm;
  float* sq = sk + TT * DK;
  float* sg = sq + TT * DK;                       // delta only
  float* sv = sg + (DELTA ? TT * DK : 0);
  float* so = sv + TT * p.dvp;
  float* sx = so + TT * p.dvp;                    // memory: [4][TT] old weight, new weight, e^{-m}, n . q
  const int tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31;
  const int rg = lane >> 3, col = warp * 8 + (lane & 7);
  const int kvh = h / p.group;
  float* st = p.state + (static_cast<size_t>(slot) * p.H + h) * p.dkp * p.dvp;
  const bool fresh = p.seq.start[s] == 0;

  float S[4 * JJ];
#pragma unroll
  for (int j = 0; j < JJ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = 16 * j + 4 * rg + e;
      S[4 * j + e] = (!fresh && i < p.dkp) ? st[static_cast<size_t>(i) * p.dvp + col] : 0.f;
    }
  const float a = KIND == RETENTION ? p.decay[h] : 0.f;
  // memory: warp 0 keeps the normaliser (channel lane + 32 j) and the maximum
  constexpr int NJ = (DK + 31) / 32;
  const size_t head = static_cast<size_t>(slot < 0 ? 0 : slot) * p.H + h;
  float nrm[NJ], mx = 0.f;
  if (MEM && warp == 0) {
#pragma unroll
    for (int j = 0; j < NJ; ++j) nrm[j] = !fresh && lane + 32 * j < p.dkp ? p.n[head * p.dkp + lane + 32 * j] : 0.f;
    if (!fresh) mx = p.m[head];
  }

  for (int t0 = 0; t0 < count; t0 += TT) {
    const int nt = min(TT, count - t0);
    if (DELTA) {
      const float* q = static_cast<const float*>(p.q);
      const float* k = static_cast<const float*>(p.k);
      for (int i = tid; i < nt * DK; i += nthr) {
        const int t = i / DK, c = i % DK;
        const size_t row = row0 + t0 + t;
        const bool in = c < p.dkp;
        sq[i] = in ? q[row * p.ld_qk + kvh * p.dkp + c] : 0.f;
        sk[i] = in ? k[row * p.ld_qk + kvh * p.dkp + c] : 0.f;
        sg[i] = in ? expf(p.glog[(row * p.H + h) * p.dkp + c]) : 0.f;
      }
    } else {
      const T* q = static_cast<const T*>(p.q);
      const T* k = static_cast<const T*>(p.k);
      const int half = p.rot / 2;
      for (int i = tid; i < nt * DK; i += nthr) {
        const int t = i / DK, c = i % DK;
        const size_t row = row0 + t0 + t;
        float qv = 0.f, kv = 0.f;
        if (c < p.dkp) {
          const size_t at = row * p.ld_qk + kvh * p.dkp;
          qv = to_f(q[at + c]);
          kv = to_f(k[at + c]);
          if (c < p.rot) {
            const int f = c < half ? c : c - half;
            const float cs = p.cs[row * half + f], sn = p.sn[row * half + f];
            const int o = c < half ? c + half : c - half;
            const float sgn = c < half ? -sn : sn;
            qv = qv * cs + to_f(q[at + o]) * sgn;
            kv = kv * cs + to_f(k[at + o]) * sgn;
          }
          kv *= p.kscale;
          if (MEM) qv *= p.qscale;
        }
        sq[i] = qv;
        sk[i] = kv;
      }
    }
    if (MEM && warp == 0) {
      float2 g = make_float2(0.f, 0.f);
      if (lane < nt) {
        const size_t row = row0 + t0 + lane;
        g = memory_gates(p.zi[row * p.ld_z + h] + to_f(static_cast<const T*>(p.bi)[h]),
                         p.zf[row * p.ld_z + h] + to_f(static_cast<const T*>(p.bf)[h]), p.cap);
      }
      float old = 0.f, now = 0.f;                  // the maximum before and after this lane's token
      for (int t = 0; t < nt; ++t) {
        const float gi = __shfl_sync(0xffffffffu, g.x, t), gf = __shfl_sync(0xffffffffu, g.y, t), next = fmaxf(gf + mx, gi);
        if (lane == t) {
          old = mx;
          now = next;
        }
        mx = next;
      }
      if (lane < nt) {
        sx[lane] = expf(g.y + old - now);
        sx[TT + lane] = expf(g.x - now);
        sx[2 * TT + lane] = expf(-now);
      }
    }
    for (int i = tid; i < nt * p.dvp; i += nthr) {
      const int t = i / p.dvp, c = i % p.dvp;
      sv[i] = to_f(static_cast<const T*>(p.v)[static_cast<size_t>(row0 + t0 + t) * p.ld_v + static_cast<size_t>(h) * p.dvp + c]);
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float* kt = sk + t * DK + 4 * rg;
      const float* qt = sq + t * DK + 4 * rg;
      float u = sv[t * p.dvp + col];
      if (DELTA) {
        const float* gt = sg + t * DK + 4 * rg;
        float d0 = 0.f, d1 = 0.f;
#pragma unroll
        for (int j = 0; j < JJ; ++j) {
          const float4 g = *reinterpret_cast<const float4*>(gt + 16 * j);
          const float4 k = *reinterpret_cast<const float4*>(kt + 16 * j);
          S[4 * j] *= g.x; S[4 * j + 1] *= g.y; S[4 * j + 2] *= g.z; S[4 * j + 3] *= g.w;
          d0 = fmaf(S[4 * j], k.x, d0);
          d1 = fmaf(S[4 * j + 1], k.y, d1);
          d0 = fmaf(S[4 * j + 2], k.z, d0);
          d1 = fmaf(S[4 * j + 3], k.w, d1);
        }
        float d = d0 + d1;
        d += __shfl_xor_sync(0xffffffffu, d, 8);
        d += __shfl_xor_sync(0xffffffffu, d, 16);
        u = p.beta[static_cast<size_t>(row0 + t0 + t) * p.H + h] * (u - d);
      }
      float o0 = 0.f, o1 = 0.f;
      const float w = MEM ? sx[t] : a;
      if (MEM) u *= sx[TT + t];
#pragma unroll
      for (int j = 0; j < JJ; ++j) {
        const float4 k = *reinterpret_cast<const float4*>(kt + 16 * j);
        const float4 q = *reinterpret_cast<const float4*>(qt + 16 * j);
        if (DELTA) {
          S[4 * j] = fmaf(k.x, u, S[4 * j]);
          S[4 * j + 1] = fmaf(k.y, u, S[4 * j + 1]);
          S[4 * j + 2] = fmaf(k.z, u, S[4 * j + 2]);
          S[4 * j + 3] = fmaf(k.w, u, S[4 * j + 3]);
        } else {
          S[4 * j] = fmaf(w, S[4 * j], k.x * u);
          S[4 * j + 1] = fmaf(w, S[4 * j + 1], k.y * u);
          S[4 * j + 2] = fmaf(w, S[4 * j + 2], k.z * u);
          S[4 * j + 3] = fmaf(w, S[4 * j + 3], k.w * u);
        }
        o0 = fmaf(S[4 * j], q.x, o0);
        o1 = fmaf(S[4 * j + 1], q.y, o1);
        o0 = fmaf(S[4 * j + 2], q.z, o0);
        o1 = fmaf(S[4 * j + 3], q.w, o1);
      }
      float o = o0 + o1;
      o += __shfl_xor_sync(0xffffffffu, o, 8);
      o += __shfl_xor_sync(0xffffffffu, o, 16);
      if (rg == 0) so[t * p.dvp + col] = o;
    }
    if (MEM && warp == 0) {
      for (int t = 0; t < nt; ++t) {
        const float w = sx[t], u = sx[TT + t];
        float d = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const int c = lane + 32 * j;
          if (c < DK) {
            nrm[j] = fmaf(w, nrm[j], u * sk[t * DK + c]);
            d = fmaf(nrm[j], sq[t * DK + c], d);
          }
        }
        d = warp_sum(d);
        if (lane == 0) sx[3 * TT + t] = d;
      }
    }
    __syncthreads();
    for (int t = warp; t < nt; t += nthr >> 5) {
      float ss = 0.f;
      for (int c = lane; c < p.dvp; c += 32) ss = fmaf(so[t * p.dvp + c], so[t * p.dvp + c], ss);
      ss = warp_sum(ss);
      const size_t row = row0 + t0 + t;
      const float inv = MEM ? 1.f / (fmaxf(fabsf(sx[3 * TT + t]), sx[2 * TT + t]) + MEMORY_EPS) : 1.f;
      float r = inv / sqrtf(ss * inv * inv / p.dv + p.eps);
      if (KIND == RETENTION && p.joint_ss) {
        r = 1.f;
        if (lane == 0) p.joint_ss[row * p.H + h] = ss;
      }
      for (int c = lane; c < p.dvp; c += 32) {
        float o = so[t * p.dvp + c] * r;
        const size_t gi = row * p.ld_gate + static_cast<size_t>(h) * p.dvp + c;
        if (DELTA) {
          if (p.norm_w) o *= to_f(static_cast<const T*>(p.norm_w)[c]);
          o *= sigmoid_t<T>(static_cast<const float*>(p.gate)[gi]);
        } else if (MEM) {
          o *= p.oscale * to_f(static_cast<const T*>(p.norm_w)[h * p.dvp + c]) * sigmoid_t<T>(to_f(static_cast<const T*>(p.gate)[gi]));
        } else if (p.joint_ss) {
          o *= to_f(static_cast<const T*>(p.norm_w)[h * p.dvp + c]) * sigmoid_t<T>(to_f(static_cast<const T*>(p.gate)[gi]));
        } else {
          o *= silu_t<T>(to_f(static_cast<const T*>(p.gate)[gi]));
        }
        static_cast<T*>(p.out)[row * p.ld_out + static_cast<size_t>(h) * p.dvp + c] = from_f<T>(o);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < JJ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = 16 * j + 4 * rg + e;
      if (i < p.dkp) st[static_cast<size_t>(i) * p.dvp + col] = S[4 * j + e];
    }
  if (MEM && warp == 0) {
#pragma unroll
    for (int j = 0; j < NJ; ++j)
      if (lane + 32 * j < p.dkp) p.n[head * p.dkp + lane + 32 * j] = nrm[j];
    if (lane == 0) p.m[head] = mx;
  }
}

// One token per sequence (the decode step), one CTA per (head, sequence).  Eight row groups of dvp / 4 threads: a thread holds
// four neighbouring value channels of every eighth key row, so a warp reads and writes whole state rows; all of a thread's
// rows are requested before the first is used.
constexpr int STEP_GROUPS = 8;

template <typename T, int J, int KIND, int MAXT>
__global__ void __launch_bounds__(MAXT, MAXT == 256 && J <= 16 ? 2 : 1) state_step_kernel(const SerialParams p) {
  constexpr bool DELTA = KIND == DELTA_RULE, MEM = KIND == MEMORY;
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.x, s = blockIdx.y;
  const int slot = p.seq.slot[s];
  if (slot < 0) return;
  const size_t row = p.seq.cu[s];
  const int DK = p.dkp, DV = p.dvp, quads = DV / 4, tid = threadIdx.x, nthr = blockDim.x;
  float* sk = sm;
  float* sq = sk + DK;
  float* sg = sq + DK;
  float* red = sg + DK;                       // [STEP_GROUPS][DV]
  float* so = red + STEP_GROUPS * DV;         // [DV], then one word per warp; memory: another per warp
  const int rg = tid / quads, col = tid % quads * 4, kvh = h / p.group;
  float* st = p.state + (static_cast<size_t>(slot) * p.H + h) * DK * DV + col;
  const bool fresh = p.seq.start[s] == 0;
  float4 S[J];
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const int i = rg + STEP_GROUPS * j;
    S[j] = !fresh && i < DK ? *reinterpret_cast<const float4*>(st + static_cast<size_t>(i) * DV) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  // memory: every thread works out the head's gates; the normaliser's channels are dealt out like the stores of k
  float w_old = 0.f, w_new = 0.f, e_neg = 0.f, mx = 0.f, nq = 0.f;
  const size_t head = static_cast<size_t>(slot) * p.H + h;
  if (MEM) {
    const float2 g = memory_gates(p.zi[row * p.ld_z + h] + to_f(static_cast<const T*>(p.bi)[h]),
                                  p.zf[row * p.ld_z + h] + to_f(static_cast<const T*>(p.bf)[h]), p.cap);
    const float m0 = fresh ? 0.f : p.m[head];
    mx = fmaxf(g.y + m0, g.x);
    w_old = expf(g.y + m0 - mx);
    w_new = expf(g.x - mx);
    e_neg = expf(-mx);
  }
  for (int c = tid; c < DK; c += nthr) {
    const size_t at = row * p.ld_qk + static_cast<size_t>(kvh) * DK;
    if (DELTA) {
      sq[c] = static_cast<const float*>(p.q)[at + c];
      sk[c] = static_cast<const float*>(p.k)[at + c];
      sg[c] = expf(p.glog[(row * p.H + h) * DK + c]);
    } else {
      const T* q = static_cast<const T*>(p.q) + at;
      const T* k = static_cast<const T*>(p.k) + at;
      float qv = to_f(q[c]), kv = to_f(k[c]);
      if (c < p.rot) {
        const int half = p.rot / 2, f = c < half ? c : c - half, o = c < half ? c + half : c - half;
        const float cs = p.cs[row * half + f], sn = c < half ? -p.sn[row * half + f] : p.sn[row * half + f];
        qv = qv * cs + to_f(q[o]) * sn;
        kv = kv * cs + to_f(k[o]) * sn;
      }
      sq[c] = MEM ? qv * p.qscale : qv;
      sk[c] = kv * p.kscale;
      if (MEM) {
        float* np = p.n + head * DK + c;
        const float nv = fmaf(w_old, fresh ? 0.f : *np, w_new * sk[c]);
        *np = nv;
        nq = fmaf(nv, sq[c], nq);
      }
    }
  }
  float4 u;
  {
    float v[4];
    const T* vp = static_cast<const T*>(p.v) + row * p.ld_v + static_cast<size_t>(h) * DV + col;
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = to_f(vp[e]);
    u = make_float4(v[0], v[1], v[2], v[3]);
  }
  __syncthreads();
  if (DELTA) {
    float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < J; ++j) {
      const int i = rg + STEP_GROUPS * j;
      if (i >= DK) break;
      const float g = sg[i], k = sk[i];
      S[j].x *= g; S[j].y *= g; S[j].z *= g; S[j].w *= g;
      d.x = fmaf(S[j].x, k, d.x); d.y = fmaf(S[j].y, k, d.y); d.z = fmaf(S[j].z, k, d.z); d.w = fmaf(S[j].w, k, d.w);
    }
    *reinterpret_cast<float4*>(red + rg * DV + col) = d;
    __syncthreads();
    float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < STEP_GROUPS; ++r) {
      const float4 x = *reinterpret_cast<const float4*>(red + r * DV + col);
      t.x += x.x; t.y += x.y; t.z += x.z; t.w += x.w;
    }
    const float b = p.beta[row * p.H + h];
    u = make_float4(b * (u.x - t.x), b * (u.y - t.y), b * (u.z - t.z), b * (u.w - t.w));
    __syncthreads();
  }
  if (MEM) {
    u.x *= w_new; u.y *= w_new; u.z *= w_new; u.w *= w_new;
  }
  const float a = DELTA ? 1.f : MEM ? w_old : p.decay[h];
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const int i = rg + STEP_GROUPS * j;
    if (i >= DK) break;
    const float k = sk[i], q = sq[i];
    S[j].x = fmaf(a, S[j].x, k * u.x); S[j].y = fmaf(a, S[j].y, k * u.y);
    S[j].z = fmaf(a, S[j].z, k * u.z); S[j].w = fmaf(a, S[j].w, k * u.w);
    *reinterpret_cast<float4*>(st + static_cast<size_t>(i) * DV) = S[j];
    o.x = fmaf(S[j].x, q, o.x); o.y = fmaf(S[j].y, q, o.y); o.z = fmaf(S[j].z, q, o.z); o.w = fmaf(S[j].w, q, o.w);
  }
  *reinterpret_cast<float4*>(red + rg * DV + col) = o;
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < DV; c += nthr) {
    float x = 0.f;
#pragma unroll
    for (int r = 0; r < STEP_GROUPS; ++r) x += red[r * DV + c];
    so[c] = x;
    ss = fmaf(x, x, ss);
  }
  ss = warp_sum(ss);
  const int warps = (nthr + 31) / 32;
  if ((tid & 31) == 0) so[DV + (tid >> 5)] = ss;
  if (MEM) {
    nq = warp_sum(nq);
    if ((tid & 31) == 0) so[DV + warps + (tid >> 5)] = nq;
  }
  __syncthreads();
  float tot = 0.f, inv = 1.f;
  for (int w = 0; w < warps; ++w) tot += so[DV + w];
  if (MEM) {
    float d = 0.f;
    for (int w = 0; w < warps; ++w) d += so[DV + warps + w];
    inv = 1.f / (fmaxf(fabsf(d), e_neg) + MEMORY_EPS);
    if (tid == 0) p.m[head] = mx;              // everyone has read the old one
  }
  float r = inv / sqrtf(tot * inv * inv / p.dv + p.eps);
  if (KIND == RETENTION && p.joint_ss) {
    r = 1.f;
    if (tid == 0) p.joint_ss[row * p.H + h] = tot;
  }
  for (int c = tid; c < DV; c += nthr) {
    float x = so[c] * r;
    const size_t gi = row * p.ld_gate + static_cast<size_t>(h) * DV + c;
    if (DELTA) {
      if (p.norm_w) x *= to_f(static_cast<const T*>(p.norm_w)[c]);
      x *= sigmoid_t<T>(static_cast<const float*>(p.gate)[gi]);
    } else if (MEM) {
      x *= p.oscale * to_f(static_cast<const T*>(p.norm_w)[h * DV + c]) * sigmoid_t<T>(to_f(static_cast<const T*>(p.gate)[gi]));
    } else if (p.joint_ss) {
      x *= to_f(static_cast<const T*>(p.norm_w)[h * DV + c]) * sigmoid_t<T>(to_f(static_cast<const T*>(p.gate)[gi]));
    } else {
      x *= silu_t<T>(to_f(static_cast<const T*>(p.gate)[gi]));
    }
    static_cast<T*>(p.out)[row * p.ld_out + static_cast<size_t>(h) * DV + c] = from_f<T>(x);
  }
}

// Input stage of the delta rule.  Grid (tiles, 2 G + H): tile = {sequence, first row, rows, offset of that row in the
// portion}, at most PREP_TILE rows.  Roles along y: G query heads, G key heads (convolution, silu, unit norm), H value heads
// (convolution, silu; the head's decays and step size).  The convolution's channels are laid out [q | k | v] in the
// projection, the taps and the state alike.  Only the portion's first tile reads the sequence's convolution state (taps - 1
// <= PREP_TILE), so that tile also replaces it, after its own reads.
constexpr int PREP_TILE = 16;
constexpr int PREP_THREADS = 128;
constexpr int PREP_MAXC = 8;   // channels a lane keeps: heads up to 256 wide

struct DeltaPrepParams {
  StateSeqs seq;
  const int* tiles;      // [n, 4]
  const void* x;         // T rows [M, ld]: q | k | v
  const void* taps;      // T [C, K]
  const void* b;         // T [M, ld]: H columns
  const float* a2;       // [M, ld_a2]: H * dkp columns
  const void* A_log;     // T [H]
  const void* dt_bias;   // T [H * dkp]
  float* conv_state;     // [slots, C, K - 1]
  float* q;              // [M, G * dkp]
  float* k;
  void* v;               // T [M, H * dvp]
  float* glog;           // [M, H * dkp]
  float* beta;           // [M, H]
  long long ld, ld_a2;
  int G, H, dk, dkp, dv, dvp, K;
  float qscale, unit_eps;
};

template <typename T>
__global__ void __launch_bounds__(PREP_THREADS) delta_prep_kernel(const DeltaPrepParams p) {
  const int* tl = p.tiles + blockIdx.x * 4;
  const int s = tl[0], row0 = tl[1], rows = tl[2], off = tl[3];
  const int slot = s < 0 ? -1 : p.seq.slot[s];
  if (slot < 0 || rows <= 0) return;
  const int y = blockIdx.y, G = p.G, K = p.K;
  const bool is_v = y >= 2 * G;
  const int width = is_v ? p.dvp : p.dkp;
  const int c0 = is_v ? 2 * G * p.dkp + (y - 2 * G) * p.dvp : y * p.dkp;
  const int C = 2 * G * p.dkp + p.H * p.dvp;
  const bool fresh = p.seq.start[s] == 0;
  const T* x = static_cast<const T*>(p.x) + c0;
  const T* taps = static_cast<const T*>(p.taps) + static_cast<size_t>(c0) * K;
  float* cst = p.conv_state + (static_cast<size_t>(slot) * C + c0) * (K - 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  for (int t = warp; t < rows; t += PREP_THREADS / 32) {
    const size_t row = row0 + t;
    float val[PREP_MAXC], ss = 0.f;
#pragma unroll
    for (int m = 0; m < PREP_MAXC; ++m) {
      const int c = lane + 32 * m;
      val[m] = 0.f;
      if (c < width) {
        float acc = 0.f;
        for (int j = 0; j < K; ++j) {           // j tokens back
          const int at = off + t - j;           // index in the portion
          float xv = 0.f;
          if (at >= 0) xv = to_f(x[(row - j) * p.ld + c]);
          else if (!fresh) xv = cst[static_cast<size_t>(c) * (K - 1) + (K - 1 + at)];
          acc = fmaf(to_f(taps[static_cast<size_t>(c) * K + K - 1 - j]), xv, acc);
        }
        val[m] = silu_t<T>(acc);
        ss = fmaf(val[m], val[m], ss);
      }
    }
    if (is_v) {
      const int h = y - 2 * G;
#pragma unroll
      for (int m = 0; m < PREP_MAXC; ++m) {
        const int c = lane + 32 * m;
        if (c < width) static_cast<T*>(p.v)[(row * p.H + h) * p.dvp + c] = from_f<T>(val[m]);
      }
      const float A = -expf(to_f(static_cast<const T*>(p.A_log)[h]));
      for (int c = lane; c < p.dkp; c += 32) {
        const float z = p.a2[row * p.ld_a2 + static_cast<size_t>(h) * p.dkp + c] +
                        to_f(static_cast<const T*>(p.dt_bias)[h * p.dkp + c]);
        p.glog[(row * p.H + h) * p.dkp + c] = A * softplus_f(z);
      }
      if (lane == 0) p.beta[row * p.H + h] = sigmoid_f(to_f(static_cast<const T*>(p.b)[row * p.ld + h]));
    } else {
      const float r = (y < G ? p.qscale : 1.f) / sqrtf(warp_sum(ss) + p.unit_eps);
      float* dst = (y < G ? p.q : p.k) + (row * G + (y < G ? y : y - G)) * p.dkp;
#pragma unroll
      for (int m = 0; m < PREP_MAXC; ++m) {
        const int c = lane + 32 * m;
        if (c < width) dst[c] = val[m] * r;
      }
    }
  }
  if (off != 0 || K < 2) return;
  __syncthreads();
  const int count = p.seq.cu[s + 1] - p.seq.cu[s];
  for (int c = threadIdx.x; c < width; c += PREP_THREADS) {
    float* d = cst + static_cast<size_t>(c) * (K - 1);
    for (int j = 0; j < K - 1; ++j) {
      const int at = count - (K - 1) + j;
      d[j] = at >= 0 ? to_f(x[(static_cast<size_t>(row0) + at) * p.ld + c]) : (fresh ? 0.f : d[j + count]);
    }
  }
}

// The same stage with four taps, a lane per eight channels: LPH lanes hold a head, a warp walks the rows of a tile with the
// last inputs in registers.  A warp takes one job: 32 / LPH of the 2 G query and key heads, 32 / LPV value heads, or 256
// decay channels.  (Any other number of taps: the kernel above.)
template <typename T, int LPH>
__device__ __forceinline__ void prep_conv_job(const DeltaPrepParams& p, int s, int row0, int rows, int off, int head, int nheads,
                                              int c_base, int width, bool unit) {
  constexpr int K = 4;
  const int lane = threadIdx.x & 31, hd = head + lane / LPH, c = lane % LPH * 8;
  const bool in = hd < nheads && c < width;
  const int ch = c_base + (hd < nheads ? hd : 0) * width + (c < width ? c : 0);    // channel in [q | k | v]
  const int C = 2 * p.G * p.dkp + p.H * p.dvp;
  const bool fresh = p.seq.start[s] == 0;
  const T* x = static_cast<const T*>(p.x) + ch;
  float* cst = p.conv_state + (static_cast<size_t>(p.seq.slot[s]) * C + ch) * (K - 1);
  float taps[K * 8], w[K - 1][8];     // w[i]: the input i + 1 tokens back
#pragma unroll
  for (int i = 0; i < K; ++i) {
    float t[8];
    vload8(static_cast<const T*>(p.taps) + static_cast<size_t>(ch) * K + i * 8, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) taps[i * 8 + e] = t[e];
  }
#pragma unroll
  for (int i = 0; i < K - 1; ++i)
#pragma unroll
    for (int e = 0; e < 8; ++e) w[i][e] = 0.f;
  float old[8 * (K - 1)];
#pragma unroll
  for (int e = 0; e < 8 * (K - 1); ++e) old[e] = 0.f;
  if (off == 0) {
    if (!fresh) {
#pragma unroll
      for (int i = 0; i < K - 1; ++i) {
        float t[8];
        vload8(cst + i * 8, t);
#pragma unroll
        for (int e = 0; e < 8; ++e) old[i * 8 + e] = t[e];
      }
    }
#pragma unroll
    for (int i = 0; i < K - 1; ++i)
#pragma unroll
      for (int e = 0; e < 8; ++e) w[i][e] = old[e * (K - 1) + K - 2 - i];
  } else {
#pragma unroll
    for (int i = 0; i < K - 1; ++i) vload8(x + (static_cast<size_t>(row0) - 1 - i) * p.ld, w[i]);   // off >= a tile > K - 1
  }
  constexpr int AHEAD = 4;            // rows requested together
  float buf[AHEAD][8];
  for (int t = 0; t < rows; ++t) {
    const size_t row = static_cast<size_t>(row0) + t;
    if (t % AHEAD == 0) {
#pragma unroll
      for (int i = 0; i < AHEAD; ++i) vload8(x + (static_cast<size_t>(row0) + min(t + i, rows - 1)) * p.ld, buf[i]);
    }
    float cur[8], y[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (t % AHEAD == i)
#pragma unroll
        for (int e = 0; e < 8; ++e) cur[e] = buf[i][e];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float a = cur[e] * taps[e * K + K - 1];
#pragma unroll
      for (int i = 0; i < K - 1; ++i) a = fmaf(w[i][e], taps[e * K + K - 2 - i], a);
      y[e] = silu_t<T>(a);
      ss = fmaf(y[e], y[e], ss);
    }
#pragma unroll
    for (int i = K - 2; i > 0; --i)
#pragma unroll
      for (int e = 0; e < 8; ++e) w[i][e] = w[i - 1][e];
#pragma unroll
    for (int e = 0; e < 8; ++e) w[0][e] = cur[e];
    if (unit) {
      if (!in) ss = 0.f;
#pragma unroll
      for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const bool is_q = hd < p.G;
      const float r = (is_q ? p.qscale : 1.f) / sqrtf(ss + p.unit_eps);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] *= r;
      if (in) vstore8((is_q ? p.q : p.k) + (row * p.G + (is_q ? hd : hd - p.G)) * p.dkp + c, y);
    } else if (in) {
      vstore8(static_cast<T*>(p.v) + (row * p.H + hd) * p.dvp + c, y);
    }
  }
  if (off != 0 || !in) return;
  const int count = p.seq.cu[s + 1] - p.seq.cu[s];
  float nw[K - 1][8];   // [j]: the input at index count - (K - 1) + j of the portion
#pragma unroll
  for (int j = 0; j < K - 1; ++j) {
    const int at = count - (K - 1) + j;
    if (at >= 0) {
      vload8(x + (static_cast<size_t>(row0) + at) * p.ld, nw[j]);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        nw[j][e] = 0.f;
#pragma unroll
        for (int m = 0; m < K - 1; ++m)
          if (m == j + count) nw[j][e] = old[e * (K - 1) + m];
      }
    }
  }
  float flat[8 * (K - 1)];
#pragma unroll
  for (int e = 0; e < 8; ++e)
#pragma unroll
    for (int j = 0; j < K - 1; ++j) flat[e * (K - 1) + j] = nw[j][e];
#pragma unroll
  for (int i = 0; i < K - 1; ++i) {
    float t[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) t[e] = flat[i * 8 + e];
    vstore8(cst + i * 8, t);
  }
}

template <typename T, int LPH, int LPV>
__global__ void __launch_bounds__(PREP_THREADS) delta_prep_vec_kernel(const DeltaPrepParams p) {
  const int* tl = p.tiles + blockIdx.x * 4;
  const int s = tl[0], row0 = tl[1], rows = tl[2], off = tl[3];
  if (s < 0 || rows <= 0 || p.seq.slot[s] < 0) return;
  const int nq = (2 * p.G * LPH + 31) / 32, nv = (p.H * LPV + 31) / 32, lane = threadIdx.x & 31;
  int job = blockIdx.y * (PREP_THREADS / 32) + (threadIdx.x >> 5);
  if (job < nq) return prep_conv_job<T, LPH>(p, s, row0, rows, off, job * (32 / LPH), 2 * p.G, 0, p.dkp, true);
  job -= nq;
  if (job < nv) return prep_conv_job<T, LPV>(p, s, row0, rows, off, job * (32 / LPV), p.H, 2 * p.G * p.dkp, p.dvp, false);
  job -= nv;
  const int c = job * 256 + lane * 8, width = p.H * p.dkp;
  if (job == 0)
    for (int t = 0; t < rows; ++t)
      for (int h = lane; h < p.H; h += 32) {
        const size_t row = static_cast<size_t>(row0) + t;
        p.beta[row * p.H + h] = sigmoid_f(to_f(static_cast<const T*>(p.b)[row * p.ld + h]));
      }
  if (c >= width) return;
  float dt[8];
  vload8(static_cast<const T*>(p.dt_bias) + c, dt);
  const float A = -expf(to_f(static_cast<const T*>(p.A_log)[c / p.dkp]));
  constexpr int AHEAD = 4;
  for (int t0 = 0; t0 < rows; t0 += AHEAD) {
    float z[AHEAD][8];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) vload8(p.a2 + (static_cast<size_t>(row0) + min(t0 + i, rows - 1)) * p.ld_a2 + c, z[i]);
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (t0 + i >= rows) break;
#pragma unroll
      for (int e = 0; e < 8; ++e) z[i][e] = A * softplus_f(z[i][e] + dt[e]);
      vstore8(p.glog + (static_cast<size_t>(row0) + t0 + i) * width + c, z[i]);
    }
  }
}

template <typename T, int KIND>
static int launch_step(const SerialParams& p, int nseq, cudaStream_t stream) {
  const int threads = STEP_GROUPS * (p.dvp / 4);    // a multiple of 16; 32 for head sizes in steps of 16
  const size_t smem = sizeof(float) * (3 * p.dkp + (STEP_GROUPS + 1) * p.dvp + 64);
  const dim3 grid(p.H, nseq);
#define B2_STEP(JV)                                                                                          \
  do {                                                                                                       \
    auto kern = threads <= 256 ? state_step_kernel<T, JV, KIND, 256> : state_step_kernel<T, JV, KIND, 512>; \
    kern<<<grid, threads, smem, stream>>>(p);                                                                \
  } while (0)
  if (p.dkp <= 32) B2_STEP(4);
  else if (p.dkp <= 64) B2_STEP(8);
  else if (p.dkp <= 128) B2_STEP(16);
  else B2_STEP(32);
#undef B2_STEP
  B2_CHECK_LAUNCH("linear_state_step");
  return 0;
}

template <typename T, int KIND>
static int launch_serial(const SerialParams& p, int nseq, cudaStream_t stream) {
  if (p.tile == 1 && p.dvp % 16 == 0) return launch_step<T, KIND>(p, nseq, stream);
  const int JJ = p.dkp <= 16 ? 1 : p.dkp <= 32 ? 2 : p.dkp <= 64 ? 4 : p.dkp <= 128 ? 8 : 16;
  const int DK = 16 * JJ;
  const size_t smem = sizeof(float) * p.tile * ((KIND == DELTA_RULE ? 3 : 2) * DK + 2 * p.dvp + (KIND == MEMORY ? 4 : 0));
  const dim3 grid(p.H, nseq);
#define B2_SERIAL(J)                                                                                            \
  do {                                                                                                          \
    auto kern = p.dvp <= 128 ? state_serial_kernel<T, J, KIND, 512> : state_serial_kernel<T, J, KIND, 1024>;  \
    if (smem > 48 * 1024)                                                                                       \
      cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));          \
    kern<<<grid, p.dvp * 4, smem, stream>>>(p);                                                                 \
  } while (0)
  if (JJ == 1) B2_SERIAL(1);
  else if (JJ == 2) B2_SERIAL(2);
  else if (JJ == 4) B2_SERIAL(4);
  else if (JJ == 8) B2_SERIAL(8);
  else B2_SERIAL(16);
#undef B2_SERIAL
  B2_CHECK_LAUNCH("linear_state");
  return 0;
}

static bool bad_heads(const char* what, int H, int group, int dk, int dkp, int dv, int dvp, int nseq) {
  if (dkp % 8 || dvp % 8 || dkp > 256 || dvp > 256 || dk > dkp || dv > dvp || dk < 1 || dv < 1 || H < 1 || group < 1 ||
      H % group || nseq > 65535) {
    set_error("%s: head sizes up to 256 in multiples of 8 (padded) and H %% group == 0 required", what);
    return true;
  }
  return false;
}

}  // namespace b2

using namespace b2;

// joint_ss given: norm_w [H * dvp] and a sigmoid gate instead of the norm per head and the silu gate (see above).
B2_EXPORT int b2_retention_serial(const void* q, const void* k, const void* v, const void* gate, void* out, float* state,
                                  const float* decay, const float* cs, const float* sn, const int* cu, const int* start,
                                  const int* slot, int nseq, int max_rows, int H, int dk, int dkp, int dv, int dvp, int rot,
                                  long long ld_in, long long ld_out, float kscale, float eps, const void* norm_w,
                                  float* joint_ss, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (nseq <= 0) return 0;
  if (joint_ss != nullptr && norm_w == nullptr) { set_error("retention: a joint norm needs its weight"); return 10; }
  if (bad_heads("retention", H, 1, dk, dkp, dv, dvp, nseq)) return 10;
  if (rot < 0 || rot % 2 || rot > dk) { set_error("retention: rotary dims must be even and at most the head size"); return 10; }
  SerialParams p = {};
  p.seq = {cu, start, slot};
  p.q = q; p.k = k; p.v = v; p.gate = gate; p.cs = cs; p.sn = sn; p.decay = decay; p.out = out; p.state = state;
  p.norm_w = norm_w; p.joint_ss = joint_ss;
  p.ld_qk = p.ld_v = p.ld_gate = ld_in; p.ld_out = ld_out;
  p.H = H; p.group = 1; p.dk = dk; p.dkp = dkp; p.dv = dv; p.dvp = dvp; p.rot = rot; p.kscale = kscale; p.eps = eps;
  p.tile = max_rows < 16 ? (max_rows < 1 ? 1 : max_rows) : 16;
  B2_DISPATCH_T(is_f32, return (launch_serial<T, RETENTION>(p, nseq, static_cast<cudaStream_t>(stream))););
}

B2_EXPORT int b2_delta_serial(const float* q, const float* k, const void* v, const float* glog, const float* beta,
                              const float* gate, const void* norm_w, void* out, float* state, const int* cu, const int* start,
                              const int* slot, int nseq, int max_rows, int H, int G, int dk, int dkp, int dv, int dvp,
                              long long ld_gate, long long ld_out, float eps, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (nseq <= 0) return 0;
  if (G < 1 || H % G || bad_heads("gated_delta", H, H / (G > 0 ? G : 1), dk, dkp, dv, dvp, nseq)) return 10;
  SerialParams p = {};
  p.seq = {cu, start, slot};
  p.q = q; p.k = k; p.v = v; p.gate = gate; p.glog = glog; p.beta = beta; p.norm_w = norm_w; p.out = out; p.state = state;
  p.ld_qk = static_cast<long long>(G) * dkp; p.ld_v = static_cast<long long>(H) * dvp; p.ld_gate = ld_gate; p.ld_out = ld_out;
  p.H = H; p.group = H / G; p.dk = dk; p.dkp = dkp; p.dv = dv; p.dvp = dvp; p.eps = eps;
  p.tile = max_rows < 16 ? (max_rows < 1 ? 1 : max_rows) : 16;
  B2_DISPATCH_T(is_f32, return (launch_serial<T, DELTA_RULE>(p, nseq, static_cast<cudaStream_t>(stream))););
}

// zi, zf: fp32 rows of stride ld_z (H columns); n: fp32 [slots, H, dkp]; m: fp32 [slots, H]; norm_w: T [H * dvp].
B2_EXPORT int b2_memory_serial(const void* q, const void* k, const void* v, const void* gate, const float* zi, const float* zf,
                               long long ld_z, const void* bi, const void* bf, const void* norm_w, void* out, float* state, float* n,
                               float* m, const int* cu, const int* start, const int* slot, int nseq, int max_rows, int H, int dk,
                               int dkp, int dv, int dvp, long long ld_in, long long ld_out, float cap, float qscale, float oscale,
                               float eps, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (nseq <= 0) return 0;
  if (bad_heads("matrix_memory", H, 1, dk, dkp, dv, dvp, nseq)) return 10;
  if (!(cap > 0.f)) { set_error("matrix_memory: the gates' cap must be positive"); return 10; }
  SerialParams p = {};
  p.seq = {cu, start, slot};
  p.q = q; p.k = k; p.v = v; p.gate = gate; p.out = out; p.state = state; p.norm_w = norm_w;
  p.ld_qk = p.ld_v = p.ld_gate = ld_in; p.ld_out = ld_out;
  p.H = H; p.group = 1; p.dk = dk; p.dkp = dkp; p.dv = dv; p.dvp = dvp; p.kscale = 1.f; p.eps = eps;
  p.zi = zi; p.zf = zf; p.bi = bi; p.bf = bf; p.n = n; p.m = m; p.ld_z = ld_z; p.cap = cap; p.qscale = qscale; p.oscale = oscale;
  p.tile = max_rows < 16 ? (max_rows < 1 ? 1 : max_rows) : 16;
  B2_DISPATCH_T(is_f32, return (launch_serial<T, MEMORY>(p, nseq, static_cast<cudaStream_t>(stream))););
}

B2_EXPORT int b2_delta_prep(const void* x, const void* taps, const void* b, const float* a2, const void* A_log,
                            const void* dt_bias, float* conv_state, float* q, float* k, void* v, float* glog, float* beta,
                            const int* cu, const int* start, const int* slot, const int* tiles, int ntiles, int H, int G,
                            int dk, int dkp, int dv, int dvp, int K, long long ld, long long ld_a2, float qscale,
                            float unit_eps, int is_f32, void* stream) {
  b2::ensure_thread_context();
  if (ntiles <= 0) return 0;
  if (G < 1 || H % G || bad_heads("delta_prep", H, H / (G > 0 ? G : 1), dk, dkp, dv, dvp, 1)) return 10;
  if (K < 1 || K - 1 > PREP_TILE || 2 * G + H > 65535) { set_error("delta_prep: 1 to %d convolution taps", PREP_TILE + 1); return 10; }
  DeltaPrepParams p = {};
  p.seq = {cu, start, slot};
  p.tiles = tiles; p.x = x; p.taps = taps; p.b = b; p.a2 = a2; p.A_log = A_log; p.dt_bias = dt_bias; p.conv_state = conv_state;
  p.q = q; p.k = k; p.v = v; p.glog = glog; p.beta = beta; p.ld = ld; p.ld_a2 = ld_a2;
  p.G = G; p.H = H; p.dk = dk; p.dkp = dkp; p.dv = dv; p.dvp = dvp; p.K = K; p.qscale = qscale; p.unit_eps = unit_eps;
  const auto lanes = [](int w) { int l = 1; while (l * 8 < w) l *= 2; return l; };
  const int lph = lanes(dkp), lpv = lanes(dvp);
  if (K == 4 && ld % 8 == 0 && ld_a2 % 8 == 0 && lph >= 4 && lpv >= 4) {
    const int jobs = (2 * G * lph + 31) / 32 + (H * lpv + 31) / 32 + (H * dkp + 255) / 256;
    const dim3 vgrid(ntiles, (jobs + PREP_THREADS / 32 - 1) / (PREP_THREADS / 32));
    cudaStream_t st = static_cast<cudaStream_t>(stream);
#define B2_PREP_V(A, B) delta_prep_vec_kernel<T, A, B><<<vgrid, PREP_THREADS, 0, st>>>(p)
#define B2_PREP_Q(A)                                                                                        \
  do {                                                                                                      \
    if (lpv == 4) B2_PREP_V(A, 4); else if (lpv == 8) B2_PREP_V(A, 8); else if (lpv == 16) B2_PREP_V(A, 16); else B2_PREP_V(A, 32); \
  } while (0)
    B2_DISPATCH_T(is_f32, {
      if (lph == 4) B2_PREP_Q(4); else if (lph == 8) B2_PREP_Q(8); else if (lph == 16) B2_PREP_Q(16); else B2_PREP_Q(32);
    });
#undef B2_PREP_Q
#undef B2_PREP_V
    B2_CHECK_LAUNCH("delta_prep");
    return 0;
  }
  const dim3 grid(ntiles, 2 * G + H);
  B2_DISPATCH_T(is_f32, delta_prep_kernel<T><<<grid, PREP_THREADS, 0, static_cast<cudaStream_t>(stream)>>>(p););
  B2_CHECK_LAUNCH("delta_prep");
  return 0;
}
