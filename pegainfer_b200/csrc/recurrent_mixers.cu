// Recurrent mixers with a matrix state per head, for ragged batches whose requests keep their state in numbered slots:
//   * short causal convolution (+ SiLU) over time per channel, with the last taps - 1 inputs of every request as state;
//   * gated delta rule:   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q        (q, k unit vectors per head)
//     with one decay g per head, or one per head and key channel (g then scales the rows of S);
//   * gated linear attention:   S <- diag(a) S + k v^T;  o = S^T q     (one decay per head and key channel, a = logistic(.)^(1 / tau));
//   * real-gated linear recurrent unit, one scalar per channel:  S <- a S + sqrt(1 - a^2) i u,  log a = -rate r softplus(lam),
//     r and i logistic gates;  the read-out is multiplied by a GELU branch.  Affine maps compose, so a portion is scanned in parallel.
//   * xLSTM matrix memory: m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T;  n likewise with k alone;
//                          o = S^T q / (max(|n . q|, e^(-m')) + 1e-6)        (i, f soft-capped log gates, m starts at 0)
//     slot layout: S [H][dim][vdim], n [H][dim], m [H][vdim + 1] (every column keeps its own copy of the running maximum)
//   * state-space duality (scalar decay per head):  S <- e^(-e^(A_log) dt) S + dt B x^T;  y = S^T C + D x,  dt = softplus(. + dt_bias)
//     (B, C of the head's group [state], x the head's slice [vdim]; the state S [state][vdim] takes the place of [dim][vdim])
//   * per-head RMS norm of the read-out times a weight times an activation of a gate projection (or the gate first, then the norm).
// State, gates, decays, unit norms and the recurrences are fp32 whatever the element type E of the activations is.
//
// Step layout: entry e of the step owns rows [row0[e], row0[e] + len[e]) of every [tokens, features] buffer (a portion
// of a prompt or one decoded token) and the state slot slot[e]; a slot's state is `state + slot * slot_stride` floats.
// Sequence kernels: one CTA per (entry, head, slice of value columns); a column of S lives in the registers of DK / 16
// neighbouring lanes (key size padded to the template's DK), tokens run one after the other.  The delta rule and the gated linear
// attention have kernels of their own, delta_seq_kernel and gla_seq_kernel; in recurrent_seq_kernel (matrix memory, state space) all threads first bring q, k, v and the gate inputs of a
// block of 32 tokens into shared memory.  The matrix memory's normaliser n is one more column with value 1.  Latency-bound per token
// (48 FMAs and two shuffle reductions per thread, one warp per scheduler).
#include <algorithm>

#include "common.cuh"
#include "mma.cuh"
#include "typed.cuh"

namespace pk {

__device__ __forceinline__ float sigmoidf_(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplusf_(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float logsigmoidf_(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// y[t][c] = act(bias[c] + sum_j w[c][j] * x[t - (taps-1-j)][c]),  x = in + in_bias (either bias may be null; act 0: none, 1: SiLU).  Inputs
// before this step's rows come from the slot's state [taps-1][C] (oldest first; zero for a new request), which afterwards holds the last
// taps - 1 inputs (old ones move up when the portion was shorter).  One thread per (channel, `gs` consecutive tokens of one entry) with
// gs >= taps - 1: an entry's first group is the only one that reads the old state, so the same thread may replace it when it is done.
// TAPS > 0: the number of taps at compile time (the window slides through registers); 0: any number.
template <typename E, int TAPS>
__global__ void causal_conv_kernel(const E* __restrict__ in, int ld_in, const E* __restrict__ in_bias, const E* __restrict__ w, const E* __restrict__ bias,
                                   float* __restrict__ state, long slot_stride, const int* __restrict__ slot, const int* __restrict__ row0,
                                   const int* __restrict__ len, E* __restrict__ out, int ld_out, int C, int taps_any, int act, int entries, int gs) {
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int taps = TAPS > 0 ? TAPS : taps_any;
  int grp = blockIdx.y, e = 0;
  for (; e < entries; ++e) {  // the entry this group of tokens belongs to
    const int ng = (len[e] + gs - 1) / gs;
    if (grp < ng) break;
    grp -= ng;
  }
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (e == entries || c >= C) return;
  const int n = len[e], o0 = grp * gs, o1 = min(n, o0 + gs);
  const E* x = in + (size_t)row0[e] * ld_in + c;
  E* y = out + (size_t)row0[e] * ld_out + c;
  float* st = state + (size_t)slot[e] * slot_stride + c;
  const float ib = in_bias ? to_f(in_bias[c]) : 0.f, b0 = bias ? to_f(bias[c]) : 0.f;
  auto input = [&](int o) { return o >= 0 ? to_f(x[(size_t)o * ld_in]) + ib : st[(size_t)(taps - 1 + o) * C]; };
  auto finish = [&](float v) { return from_f<E>(act ? v / (1.f + expf(-v)) : v); };
  if constexpr (TAPS > 0) {
    float wr[TAPS], h[TAPS];  // h[j]: input of taps - 1 - j tokens ago
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wr[j] = to_f(w[(size_t)c * TAPS + j]);
#pragma unroll
    for (int j = 1; j < TAPS; ++j) h[j] = input(o0 - TAPS + j);
#pragma unroll 4
    for (int o = o0; o < o1; ++o) {
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) h[j] = h[j + 1];
      h[TAPS - 1] = to_f(x[(size_t)o * ld_in]) + ib;
      float acc = b0;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(wr[j], h[j], acc);
      y[(size_t)o * ld_out] = finish(acc);
    }
  } else {
    for (int o = o0; o < o1; ++o) {
      float acc = b0;
      for (int j = 0; j < taps; ++j) acc = fmaf(to_f(w[(size_t)c * taps + j]), input(o - (taps - 1) + j), acc);
      y[(size_t)o * ld_out] = finish(acc);
    }
  }
  if (grp == 0)
    for (int i = 0; i < taps - 1; ++i) {  // ascending: an old entry is read before its place is written
      const int o = n - (taps - 1) + i;
      st[(size_t)i * C] = o >= 0 ? to_f(x[(size_t)o * ld_in]) + ib : st[(size_t)(i + n) * C];
    }
}

struct SeqArgs {
  const void* qkv;     // [tokens, ld]: q at q_off + kv_head * dim, k at k_off + kv_head * dim, v at v_off + head * vdim
  int ld, q_off, k_off, v_off;
  const float* z;      // [tokens, ldz] fp32 few-row projections: z[za_off + head], z[zb_off + head]
  int ldz, za_off, zb_off;
  const float* p0;     // delta: A_log [H];  matrix memory: input-gate bias [H]
  const float* p1;     // delta: dt_bias [H];  matrix memory: forget-gate bias [H]
  float* state;        // slot base (this layer's block)
  long slot_stride;
  const int *slot, *row0, *len;
  float* out;          // [tokens, H * vdim] fp32 read-out
  float* den;          // matrix memory: [tokens, H] divisor
  int H, G, dim, vdim;
  float cap;           // matrix memory: gate soft cap
  const void* dt;      // state space: [tokens, ld_dt] element type, step-size projection of head h at dt_off + h
  int ld_dt, dt_off;
  const float* p2;     // state space: skip weight D [H]  (p0 = A_log, p1 = dt_bias)
  const float* zc;     // delta rule with a decay per key channel: [tokens, ld_zc], pre-activation of (head, channel) at h * dim + d; p1 = dt_bias [H * dim]
  int ld_zc;
  int zc_ready;        // 1: zc holds the decays themselves
};

// MODE 1: xLSTM matrix memory.  MODE 2: state-space duality (q = C, k = B, v = x; dim = state size).
// Thread layout: KS = DK / 16 neighbouring lanes share one state column, each holding 16 of its DK entries in registers
// (entry (m * KS + ks) * 4 + e for m < 4, e < 4, so that the lanes' 16-byte reads of k / q from shared memory fall on
// consecutive banks); the two dot products per token are finished with log2(KS) shuffles.  128 / KS columns per CTA; the
// matrix memory's normaliser column rides in one more warp of the head's first CTA.
template <typename E, int DK, int MODE>
__global__ void __launch_bounds__(160) recurrent_seq_kernel(SeqArgs a) {
  constexpr int KS = DK / 16, COLS = 128 / KS, TB = DK <= 128 ? 32 : 16, NS = 16;  // NS state entries per thread
  __shared__ __align__(16) float ks[TB][DK];
  __shared__ __align__(16) float qs[TB][DK];
  __shared__ float vs[TB][COLS];
  __shared__ float g0[TB], g1[TB];  // memory: log forget gate, log input gate;  state space: decay, step size
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int e = blockIdx.x, h = blockIdx.y, kvh = h / (a.H / a.G);
  const int tid = threadIdx.x, warp = tid >> 5;
  const int n = a.len[e], r0 = a.row0[e], dim = a.dim, vdim = a.vdim;
  const int cl = tid / KS, ksi = tid % KS;  // column inside the CTA, share of the key axis
  const int col0 = blockIdx.z * COLS, col = col0 + cl;
  const bool is_v = tid < 128 && col < vdim;
  const bool is_n = MODE == 1 && blockIdx.z == 0 && tid >= 128 && tid < 128 + KS;
  float* base = a.state + (size_t)a.slot[e] * a.slot_stride;
  float* S_g = base + (size_t)h * dim * vdim;                      // [dim][vdim]
  float* n_g = base + (size_t)a.H * dim * vdim + (size_t)h * dim;  // matrix memory only
  // one copy of the running maximum per column: CTAs of a head never read what another one wrote
  float* m_g = base + (size_t)a.H * dim * vdim + (size_t)a.H * dim + (size_t)h * (vdim + 1) + (is_v ? col : vdim);
  float S[NS];
#pragma unroll
  for (int j = 0; j < NS; ++j) {
    const int i = ((j >> 2) * KS + ksi) * 4 + (j & 3);
    S[j] = i < dim ? (is_v ? S_g[(size_t)i * vdim + col] : (is_n ? n_g[i] : 0.f)) : 0.f;
  }
  float m = (MODE == 1 && (is_v || is_n)) ? m_g[0] : 0.f;
  const E* X = static_cast<const E*>(a.qkv);
  const float qscale = 1.f / sqrtf((float)dim);
  const size_t out_ld = (size_t)a.H * vdim;
  for (int b0 = 0; b0 < n; b0 += TB) {
    const int nb = min(TB, n - b0);
    __syncthreads();  // the previous block's readers are done
    // 1. raw q, k, v and gate inputs of the block's tokens (independent loads, many in flight)
    const E* Xb = X + (size_t)(r0 + b0) * a.ld;
    bool staged = false;
    if constexpr (sizeof(E) == 2) {
      // 16-byte pieces of 8 bf16 when every row slice starts on a 16-byte boundary
      const int qo = a.q_off + kvh * dim, ko = a.k_off + kvh * dim, vo = a.v_off + h * vdim + col0;
      if (((a.ld | qo | ko | vo | dim | vdim) & 7) == 0 && (reinterpret_cast<uintptr_t>(X) & 15) == 0) {
        staged = true;
        constexpr int PR = DK / 8;
        for (int i = tid; i < nb * PR; i += blockDim.x) {
          const int tt = i / PR, d0 = (i % PR) * 8;
          const E* row = Xb + (size_t)tt * a.ld;
          uint4 qv = make_uint4(0, 0, 0, 0), kv = qv;
          if (d0 < dim) {
            qv = *reinterpret_cast<const uint4*>(row + qo + d0);
            kv = *reinterpret_cast<const uint4*>(row + ko + d0);
          }
          *reinterpret_cast<float4*>(&qs[tt][d0]) = make_float4(bf16_lo(qv.x), bf16_hi(qv.x), bf16_lo(qv.y), bf16_hi(qv.y));
          *reinterpret_cast<float4*>(&qs[tt][d0 + 4]) = make_float4(bf16_lo(qv.z), bf16_hi(qv.z), bf16_lo(qv.w), bf16_hi(qv.w));
          *reinterpret_cast<float4*>(&ks[tt][d0]) = make_float4(bf16_lo(kv.x), bf16_hi(kv.x), bf16_lo(kv.y), bf16_hi(kv.y));
          *reinterpret_cast<float4*>(&ks[tt][d0 + 4]) = make_float4(bf16_lo(kv.z), bf16_hi(kv.z), bf16_lo(kv.w), bf16_hi(kv.w));
        }
        constexpr int PV = COLS / 8;
        for (int i = tid; i < nb * PV; i += blockDim.x) {
          const int tt = i / PV, c0 = (i % PV) * 8;
          uint4 vv = make_uint4(0, 0, 0, 0);
          if (col0 + c0 < vdim) vv = *reinterpret_cast<const uint4*>(Xb + (size_t)tt * a.ld + vo + c0);
          vs[tt][c0] = bf16_lo(vv.x), vs[tt][c0 + 1] = bf16_hi(vv.x), vs[tt][c0 + 2] = bf16_lo(vv.y), vs[tt][c0 + 3] = bf16_hi(vv.y);
          vs[tt][c0 + 4] = bf16_lo(vv.z), vs[tt][c0 + 5] = bf16_hi(vv.z), vs[tt][c0 + 6] = bf16_lo(vv.w), vs[tt][c0 + 7] = bf16_hi(vv.w);
        }
      }
    }
#pragma unroll 4
    for (int i = staged ? nb * DK : tid; i < nb * DK; i += blockDim.x) {
      const int tt = i / DK, d = i % DK;
      const E* row = Xb + (size_t)tt * a.ld;
      qs[tt][d] = d < dim ? to_f(row[a.q_off + kvh * dim + d]) : 0.f;
      ks[tt][d] = d < dim ? to_f(row[a.k_off + kvh * dim + d]) : 0.f;
    }
#pragma unroll 4
    for (int i = staged ? nb * COLS : tid; i < nb * COLS; i += blockDim.x) {
      const int tt = i / COLS, c = i % COLS;
      vs[tt][c] = col0 + c < vdim ? to_f(Xb[(size_t)tt * a.ld + a.v_off + h * vdim + col0 + c]) : 0.f;
    }
    if (MODE == 2) {
      if (tid < nb) {  // step size and decay of the head at this token, from the projection's output
        const float step = softplusf_(to_f(static_cast<const E*>(a.dt)[(size_t)(r0 + b0 + tid) * a.ld_dt + a.dt_off + h]) + a.p1[h]);
        g0[tid] = expf(-expf(a.p0[h]) * step);
        g1[tid] = step;
      }
    } else if (tid < nb) {
      const size_t row = (size_t)(r0 + b0 + tid);
      const float za = a.z[row * a.ldz + a.za_off + h], zb = a.z[row * a.ldz + a.zb_off + h];  // forget gate, input gate
      g0[tid] = logsigmoidf_(a.cap * tanhf((za + a.p1[h]) / a.cap));
      g1[tid] = a.cap * tanhf((zb + a.p0[h]) / a.cap);
    }
    __syncthreads();
    // 2. the query's scale
    if (MODE == 1)
      for (int i = tid; i < nb * DK; i += blockDim.x) qs[i / DK][i % DK] *= qscale;
    __syncthreads();
    if (warp >= 4 && !(MODE == 1 && blockIdx.z == 0)) continue;  // the extra warp only carries the normaliser
    // 3. the recurrence, token by token (whole warps run it: the shuffles below need every lane)
#pragma unroll 2
    for (int tt = 0; tt < nb; ++tt) {
      const size_t row = (size_t)(r0 + b0 + tt);
      const float vt = tid < 128 ? vs[tt][cl] : 1.f;
      const float4* k4p = reinterpret_cast<const float4*>(&ks[tt][0]) + ksi;
      const float4* q4p = reinterpret_cast<const float4*>(&qs[tt][0]) + ksi;
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
      if (MODE == 2) {
        const float fa = g0[tt], wb = g1[tt] * vt;
#pragma unroll
        for (int mi = 0; mi < NS / 4; ++mi) {
          const float4 k4 = k4p[mi * KS];
          const float4 q4 = q4p[mi * KS];
          S[mi * 4] = fmaf(k4.x, wb, fa * S[mi * 4]);
          S[mi * 4 + 1] = fmaf(k4.y, wb, fa * S[mi * 4 + 1]);
          S[mi * 4 + 2] = fmaf(k4.z, wb, fa * S[mi * 4 + 2]);
          S[mi * 4 + 3] = fmaf(k4.w, wb, fa * S[mi * 4 + 3]);
          o0 = fmaf(S[mi * 4], q4.x, o0);
          o1 = fmaf(S[mi * 4 + 1], q4.y, o1);
          o2 = fmaf(S[mi * 4 + 2], q4.z, o2);
          o3 = fmaf(S[mi * 4 + 3], q4.w, o3);
        }
        float o = (o0 + o1) + (o2 + o3);
#pragma unroll
        for (int s = 1; s < KS; s <<= 1) o += __shfl_xor_sync(0xffffffffu, o, s);
        if (is_v && ksi == 0) a.out[row * out_ld + h * vdim + col] = fmaf(a.p2[h], vt, o);
      } else {
        const float f = g0[tt], ig = g1[tt];
        const float mn = fmaxf(f + m, ig);
        const float fa = expf(f + m - mn), wb = expf(ig - mn) * vt;
        m = mn;
#pragma unroll
        for (int mi = 0; mi < NS / 4; ++mi) {
          const float4 k4 = k4p[mi * KS];
          const float4 q4 = q4p[mi * KS];
          S[mi * 4] = fmaf(k4.x, wb, fa * S[mi * 4]);
          S[mi * 4 + 1] = fmaf(k4.y, wb, fa * S[mi * 4 + 1]);
          S[mi * 4 + 2] = fmaf(k4.z, wb, fa * S[mi * 4 + 2]);
          S[mi * 4 + 3] = fmaf(k4.w, wb, fa * S[mi * 4 + 3]);
          o0 = fmaf(S[mi * 4], q4.x, o0);
          o1 = fmaf(S[mi * 4 + 1], q4.y, o1);
          o2 = fmaf(S[mi * 4 + 2], q4.z, o2);
          o3 = fmaf(S[mi * 4 + 3], q4.w, o3);
        }
        float o = (o0 + o1) + (o2 + o3);
#pragma unroll
        for (int s = 1; s < KS; s <<= 1) o += __shfl_xor_sync(0xffffffffu, o, s);
        if (is_v && ksi == 0) a.out[row * out_ld + h * vdim + col] = o;
        else if (is_n && ksi == 0) a.den[row * a.H + h] = fmaxf(fabsf(o), expf(-mn)) + 1e-6f;
      }
    }
  }
  if (is_v || is_n) {
#pragma unroll
    for (int j = 0; j < NS; ++j) {
      const int i = ((j >> 2) * KS + ksi) * 4 + (j & 3);
      if (i < dim) {
        if (is_v) S_g[(size_t)i * vdim + col] = S[j];
        else n_g[i] = S[j];
      }
    }
    if (MODE == 1 && ksi == 0) m_g[0] = m;
  }
}

// ---- gated delta rule.  CTA = (entry, head, COLS value columns), warp-specialised: warps 0-3 run the recurrence, warps 4-7 prepare the next
// TB tokens meanwhile (unit vectors, gates, k . q) in the other of two shared-memory stages; one barrier per TB tokens.
// Recurrence: KS = DK / 16 neighbouring lanes share one state column, 16 entries each as eight packed pairs (two-wide fp32 arithmetic), entry
// (m * KS + ks) * 4 + e for m < 4, e < 4, so that the lanes' 16-byte shared-memory reads fall on consecutive banks.  Both products of a
// token are taken on the decayed state before the write, o = S^T q = (g S)^T q + (k . q) u, so that their reductions over the lanes overlap and
// only one of them is on the path to the next token.  CH: one decay per key channel (a third vector per token), else one per head.
struct F2 {  // a packed pair of floats
  unsigned long long v;
};
__device__ __forceinline__ F2 f2_mul(F2 a, F2 b) {
  F2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v));
  return r;
}
__device__ __forceinline__ F2 f2_add(F2 a, F2 b) {
  F2 r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v));
  return r;
}
__device__ __forceinline__ F2 f2_fma(F2 a, F2 b, F2 c) {
  F2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r.v) : "l"(a.v), "l"(b.v), "l"(c.v));
  return r;
}
__device__ __forceinline__ F2 f2_pack(float lo, float hi) {
  F2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r.v) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 f2_unpack(F2 a) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(a.v));
  return r;
}

constexpr int kDeltaTB = 16;  // tokens per stage
template <int DK, bool CH>
constexpr int delta_stage_floats() {
  return kDeltaTB * (2 * DK + 128 / (DK / 16) + (CH ? DK : 0) + 4);
}

template <typename E, int DK, bool CH>
__global__ void __launch_bounds__(256) delta_seq_kernel(SeqArgs a) {
  constexpr int KS = DK / 16, COLS = 128 / KS, TB = kDeltaTB, NV = DK / 32, TW = TB / 4;  // TW: tokens a preparing warp handles per stage
  extern __shared__ __align__(16) float ds_sm[];
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int e = blockIdx.x, h = blockIdx.y, kvh = h / (a.H / a.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n = a.len[e], r0 = a.row0[e], dim = a.dim, vdim = a.vdim, col0 = blockIdx.z * COLS;
  const int n_stages = (n + TB - 1) / TB;
  auto ks_of = [&](int b) { return ds_sm + (b & 1) * delta_stage_floats<DK, CH>(); };  // k [TB][DK] | q [TB][DK] | v [TB][COLS] | scalars [4][TB] | decays [TB][DK]
  constexpr int QO = TB * DK, VO = 2 * TB * DK, SO = VO + TB * COLS, GO = SO + 4 * TB;
  if (warp >= 4) {
    // ---- preparation
    const E* X = static_cast<const E*>(a.qkv);
    const int qo = a.q_off + kvh * dim, ko = a.k_off + kvh * dim, vo = a.v_off + h * vdim + col0, pw = warp - 4, d0 = lane * NV;
    const float qscale = 1.f / sqrtf((float)dim), rate = expf(a.p0[h]);
    // Raw inputs of a stage wait in registers from one barrier to the next, so that their loads' latency is hidden: fetch() issues the loads
    // of a stage, finish() turns them into what the recurrence reads.
    constexpr int NW = sizeof(E) == 2 ? (NV + 1) / 2 : NV, VPT = TB * COLS / 128;  // 32-bit words per head row and lane; values per thread
    const bool vec = ((a.ld | qo | ko | dim) & (NV - 1)) == 0 && (reinterpret_cast<uintptr_t>(X) & (sizeof(E) * NV - 1)) == 0;
    uint32_t qr[TW][NW], kr[TW][NW];
    float gr[CH ? TW : 1][NV];
    E vr[VPT];
    float za = 0.f, zb = 0.f;
    const int pt = tid - 128;
    auto load_row = [&](const E* p, uint32_t* w) {  // entries d0 .. d0 + NV - 1 of a head's row (zero from dim on)
#pragma unroll
      for (int i = 0; i < NW; ++i) w[i] = 0u;
      if (vec && NV > 1) {
        if (d0 >= dim) return;
        if constexpr (NW == 1) w[0] = *reinterpret_cast<const uint32_t*>(p + d0);
        else if constexpr (NW == 2) *reinterpret_cast<uint2*>(w) = *reinterpret_cast<const uint2*>(p + d0);
        else {
#pragma unroll
          for (int i = 0; i < NW / 4; ++i) *reinterpret_cast<uint4*>(w + 4 * i) = *reinterpret_cast<const uint4*>(reinterpret_cast<const uint32_t*>(p + d0) + 4 * i);
        }
      } else {
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          if (d0 + j >= dim) continue;
          if constexpr (sizeof(E) == 2) w[j / 2] |= (uint32_t)*reinterpret_cast<const uint16_t*>(p + d0 + j) << (16 * (j & 1));
          else w[j] = *reinterpret_cast<const uint32_t*>(p + d0 + j);
        }
      }
    };
    auto word = [&](const uint32_t* w, int j) {
      if constexpr (sizeof(E) == 2) return j & 1 ? bf16_hi(w[j / 2]) : bf16_lo(w[j / 2]);
      else return __uint_as_float(w[j]);
    };
    auto fetch = [&](int b) {
      const int t0 = b * TB, nb = min(TB, n - t0);
#pragma unroll
      for (int i = 0; i < TW; ++i) {
        const int tt = min(pw + 4 * i, nb - 1);  // past the end: the last token once more (never read)
        const E* row = X + (size_t)(r0 + t0 + tt) * a.ld;
        load_row(row + qo, qr[i]);
        load_row(row + ko, kr[i]);
        if constexpr (CH) {
#pragma unroll
          for (int j = 0; j < NV; ++j) gr[i][j] = d0 + j < dim ? a.zc[(size_t)(r0 + t0 + tt) * a.ld_zc + h * dim + d0 + j] : 0.f;
        }
      }
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int at = pt + 128 * i, tt = min(at / COLS, nb - 1), c = at % COLS;
        vr[i] = col0 + c < vdim ? X[(size_t)(r0 + t0 + tt) * a.ld + vo + c] : from_f<E>(0.f);
      }
      if (pw == 0 && lane < nb) {
        const float* z = a.z + (size_t)(r0 + t0 + lane) * a.ldz;
        if (!CH) za = z[a.za_off + h];
        zb = z[a.zb_off + h];
      }
    };
    auto finish = [&](int b) {
      float* sm = ks_of(b);
      float qq[TW], kk[TW], kq[TW];
#pragma unroll
      for (int i = 0; i < TW; ++i) {
        qq[i] = kk[i] = kq[i] = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          const float q = word(qr[i], j), k = word(kr[i], j);
          qq[i] = fmaf(q, q, qq[i]);
          kk[i] = fmaf(k, k, kk[i]);
          kq[i] = fmaf(k, q, kq[i]);
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < TW; ++i) {
          qq[i] += __shfl_xor_sync(0xffffffffu, qq[i], o);
          kk[i] += __shfl_xor_sync(0xffffffffu, kk[i], o);
          kq[i] += __shfl_xor_sync(0xffffffffu, kq[i], o);
        }
#pragma unroll
      for (int i = 0; i < TW; ++i) {
        const int tt = pw + 4 * i;
        const float qf = qscale / sqrtf(qq[i] + 1e-6f), kf = 1.f / sqrtf(kk[i] + 1e-6f);
        if (lane == 0) sm[SO + 2 * TB + tt] = kq[i] * qf * kf;
        float kd[NV], qd[NV];
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          kd[j] = word(kr[i], j) * kf;
          qd[j] = word(qr[i], j) * qf;
        }
        float gd[NV];
        if constexpr (CH) {
#pragma unroll
          for (int j = 0; j < NV; ++j) {
            gd[j] = gr[i][j];
            if (d0 + j >= dim) gd[j] = 1.f;
            else if (!a.zc_ready) gd[j] = expf(-rate * softplusf_(gd[j] + a.p1[h * dim + d0 + j]));
          }
        }
        if constexpr (NV >= 4) {
#pragma unroll
          for (int j = 0; j < NV; j += 4) {
            *reinterpret_cast<float4*>(sm + tt * DK + d0 + j) = make_float4(kd[j], kd[j + 1], kd[j + 2], kd[j + 3]);
            *reinterpret_cast<float4*>(sm + QO + tt * DK + d0 + j) = make_float4(qd[j], qd[j + 1], qd[j + 2], qd[j + 3]);
            if constexpr (CH) *reinterpret_cast<float4*>(sm + GO + tt * DK + d0 + j) = make_float4(gd[j], gd[j + 1], gd[j + 2], gd[j + 3]);
          }
        } else {
#pragma unroll
          for (int j = 0; j < NV; ++j) {
            sm[tt * DK + d0 + j] = kd[j];
            sm[QO + tt * DK + d0 + j] = qd[j];
            if constexpr (CH) sm[GO + tt * DK + d0 + j] = gd[j];
          }
        }
      }
#pragma unroll
      for (int i = 0; i < VPT; ++i) sm[VO + pt + 128 * i] = to_f(vr[i]);
      if (pw == 0 && lane < TB) {
        if (!CH) sm[SO + lane] = expf(-rate * softplusf_(za + a.p1[h]));
        sm[SO + TB + lane] = sigmoidf_(zb);
      }
    };
    fetch(0);
    finish(0);
    if (n_stages > 1) fetch(1);
    for (int b = 0; b < n_stages; ++b) {
      __syncthreads();  // stage b is complete, and nobody reads the other one any more
      if (b + 1 < n_stages) {
        finish(b + 1);
        if (b + 2 < n_stages) fetch(b + 2);
      }
    }
    return;
  }
  // ---- recurrence
  const int cl = tid / KS, ksi = tid % KS, col = col0 + cl;
  const bool on = col < vdim;
  float* S_g = a.state + (size_t)a.slot[e] * a.slot_stride + (size_t)h * dim * vdim;  // [dim][vdim]
  F2 S[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int i = ((j >> 1) * KS + ksi) * 4 + (j & 1) * 2;
    S[j] = f2_pack(on && i < dim ? S_g[(size_t)i * vdim + col] : 0.f, on && i + 1 < dim ? S_g[(size_t)(i + 1) * vdim + col] : 0.f);
  }
  const size_t out_ld = (size_t)a.H * vdim;
  float* out = a.out + (size_t)r0 * out_ld + h * vdim + col;
  for (int b = 0; b < n_stages; ++b) {
    __syncthreads();
    const float* sm = ks_of(b);
    const int nb = min(TB, n - b * TB);
#pragma unroll 4
    for (int tt = 0; tt < nb; ++tt) {
      const ulonglong2* kp = reinterpret_cast<const ulonglong2*>(sm + tt * DK) + ksi;
      const ulonglong2* qp = reinterpret_cast<const ulonglong2*>(sm + QO + tt * DK) + ksi;
      const ulonglong2* gp = reinterpret_cast<const ulonglong2*>(sm + GO + tt * DK) + ksi;
      const float vt = sm[VO + tt * COLS + cl], beta = sm[SO + TB + tt], kq = sm[SO + 2 * TB + tt];
      const F2 g1 = CH ? F2{0} : f2_pack(sm[SO + tt], sm[SO + tt]);
      F2 kk[8], c0{0}, c1{0}, o0{0}, o1{0};
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const ulonglong2 k2 = kp[m * KS], q2 = qp[m * KS];
        kk[2 * m].v = k2.x;
        kk[2 * m + 1].v = k2.y;
        if constexpr (CH) {
          const ulonglong2 g2 = gp[m * KS];
          S[2 * m] = f2_mul(S[2 * m], F2{g2.x});
          S[2 * m + 1] = f2_mul(S[2 * m + 1], F2{g2.y});
        } else {
          S[2 * m] = f2_mul(S[2 * m], g1);
          S[2 * m + 1] = f2_mul(S[2 * m + 1], g1);
        }
        c0 = f2_fma(S[2 * m], kk[2 * m], c0);
        c1 = f2_fma(S[2 * m + 1], kk[2 * m + 1], c1);
        o0 = f2_fma(S[2 * m], F2{q2.x}, o0);
        o1 = f2_fma(S[2 * m + 1], F2{q2.y}, o1);
      }
      const float2 c2 = f2_unpack(f2_add(c0, c1)), o2 = f2_unpack(f2_add(o0, o1));
      float kv = c2.x + c2.y, o = o2.x + o2.y;
#pragma unroll
      for (int s = 1; s < KS; s <<= 1) {
        kv += __shfl_xor_sync(0xffffffffu, kv, s);
        o += __shfl_xor_sync(0xffffffffu, o, s);
      }
      const float u = beta * (vt - kv);
      const F2 u2 = f2_pack(u, u);
#pragma unroll
      for (int j = 0; j < 8; ++j) S[j] = f2_fma(kk[j], u2, S[j]);
      if (on && ksi == 0) out[(size_t)(b * TB + tt) * out_ld] = fmaf(kq, u, o);
    }
  }
  if (on) {
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int i = ((j >> 1) * KS + ksi) * 4 + (j & 1) * 2;
      const float2 v = f2_unpack(S[j]);
      if (i < dim) S_g[(size_t)i * vdim + col] = v.x;
      if (i + 1 < dim) S_g[(size_t)(i + 1) * vdim + col] = v.y;
    }
  }
}

template <typename E, int DK, bool CH>
static void launch_delta_t(const SeqArgs& a, int entries, cudaStream_t st) {
  constexpr int COLS = 128 / (DK / 16);
  constexpr size_t need = 2 * delta_stage_floats<DK, CH>() * sizeof(float), apart = 116 * 1024;
  const dim3 g(entries, a.H, (a.vdim + COLS - 1) / COLS);
  // the chain of tokens sets the time, so two CTAs never share an SM while there is one for each: a programmatic launch would otherwise place
  // them wherever the previous kernel's CTAs have just left
  const size_t smem = (long)g.x * g.y * g.z <= sm_count() ? (need > apart ? need : apart) : need;
  static bool attr_set = false;  // per template instance
  if (!attr_set) {
    cudaFuncSetAttribute(delta_seq_kernel<E, DK, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(need > apart ? need : apart));
    attr_set = true;
  }
  launch(delta_seq_kernel<E, DK, CH>, g, dim3(256), smem, st, true, a);
}
template <typename E, bool CH>
static int launch_delta(const SeqArgs& a, int entries, cudaStream_t st) {
  if (a.dim > 256) return -2;
  if (a.dim <= 32) launch_delta_t<E, 32, CH>(a, entries, st);
  else if (a.dim <= 64) launch_delta_t<E, 64, CH>(a, entries, st);
  else if (a.dim <= 128) launch_delta_t<E, 128, CH>(a, entries, st);
  else launch_delta_t<E, 256, CH>(a, entries, st);
  return (int)cudaGetLastError();
}

// ---- gated linear attention.  CTA = (entry, head, COLS value columns), warp-specialised: warps 0-3 run the recurrence over stages of TB tokens,
// warps 4-7 keep kStages of them on their way into shared memory (as stored; cp.async where the rows are laid out for it) and add up read-outs.
// Recurrence: KL = DK / RK neighbouring lanes share RC state columns, RK key entries of each (RK * RC = 16, packed pairs along the key axis), so
// that every read of k, q and the decays from shared memory serves RC columns.  A read-out is a sum over those lanes that no later token waits
// for: every thread leaves its share in shared memory, and warps 4-7 add the shares of a stage while the recurrence runs the next one.
struct GlaArgs {
  const void* qkv;     // [tokens, ld]: q at q_off + head * dim, k at k_off + head * dim, v at v_off + head * vdim
  int ld, q_off, k_off, v_off;
  const float* zc;     // [tokens, ld_zc]: pre-activation of the decay of (head, channel) at h * dim + d, or the decay itself (ready)
  int ld_zc, ready;
  const float* bias;   // [H * dim]
  float inv_tau;
  float* state;
  long slot_stride;
  const int *slot, *row0, *len;
  float* out;          // [tokens, H * vdim]
  int H, dim, vdim;
};
__device__ __forceinline__ float logistic_decay(float z, float inv_tau) { return expf(logsigmoidf_(z) * inv_tau); }

template <typename E, int DK>
struct GlaTile {
  static constexpr int TB = 16, COLS = 128 / (DK / 16), RK = DK <= 128 ? 4 : 8, RC = 16 / RK, KL = DK / RK, kStages = sizeof(E) == 2 ? 4 : 3;
  // bytes of a stage: k [TB][DK] | q [TB][DK] | v [TB][COLS] in the element type, decays [TB][DK] fp32
  static constexpr int kQ = TB * DK * sizeof(E), kV = 2 * kQ, kG = kV + TB * COLS * sizeof(E), kStage = kG + TB * DK * 4;
  static constexpr int kShares = TB * 128 * RC;  // floats of a stage's read-out shares: [TB][128 threads][RC]
  static constexpr size_t kSmem = (size_t)kStages * kStage + 2 * kShares * sizeof(float);
};
// two packed pairs = four consecutive entries
__device__ __forceinline__ void ld_pairs(const float* p, F2* o) {
  const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
  o[0].v = v.x;
  o[1].v = v.y;
}
__device__ __forceinline__ void ld_pairs(const bf16* p, F2* o) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  o[0] = f2_pack(bf16_lo(v.x), bf16_hi(v.x));
  o[1] = f2_pack(bf16_lo(v.y), bf16_hi(v.y));
}
template <int N>
__device__ __forceinline__ void ld_run(const float* p, float* o) {
  if constexpr (N == 4) *reinterpret_cast<float4*>(o) = *reinterpret_cast<const float4*>(p);
  else *reinterpret_cast<float2*>(o) = *reinterpret_cast<const float2*>(p);
}
template <int N>
__device__ __forceinline__ void ld_run(const bf16* p, float* o) {
  uint32_t u[N / 2];
  if constexpr (N == 4) *reinterpret_cast<uint2*>(u) = *reinterpret_cast<const uint2*>(p);
  else u[0] = *reinterpret_cast<const uint32_t*>(p);
#pragma unroll
  for (int i = 0; i < N / 2; ++i) {
    o[2 * i] = bf16_lo(u[i]);
    o[2 * i + 1] = bf16_hi(u[i]);
  }
}
// GT tokens of the recurrence; their shares are stored after the last one, so that the loads of all of them may be under way together
constexpr int kGlaGroup = 4;
template <typename E, int DK, int GT>
__device__ __forceinline__ void gla_tokens(F2 (&S)[GlaTile<E, DK>::RC][GlaTile<E, DK>::RK / 2], const unsigned char* sm, float* share, int t0, int ksl, int cl) {
  typedef GlaTile<E, DK> L;
  constexpr int RK = L::RK, RC = L::RC;
  const E* ks = reinterpret_cast<const E*>(sm) + 4 * ksl;
  const E* qs = reinterpret_cast<const E*>(sm + L::kQ) + 4 * ksl;
  const E* vs = reinterpret_cast<const E*>(sm + L::kV) + cl;
  const float* gs = reinterpret_cast<const float*>(sm + L::kG) + 4 * ksl;
  float r[GT][RC];
#pragma unroll
  for (int t = 0; t < GT; ++t) {
    const int tt = t0 + t;
    F2 vc[RC];
    float v[RC];
    ld_run<RC>(vs + tt * L::COLS, v);
#pragma unroll
    for (int c = 0; c < RC; ++c) vc[c] = f2_pack(v[c], v[c]);
    F2 o[RC];
#pragma unroll
    for (int m = 0; m < RK / 4; ++m) {
      F2 k[2], q[2], g[2];
      ld_pairs(ks + tt * DK + m * 4 * L::KL, k);
      ld_pairs(qs + tt * DK + m * 4 * L::KL, q);
      ld_pairs(gs + tt * DK + m * 4 * L::KL, g);
#pragma unroll
      for (int c = 0; c < RC; ++c) {
        S[c][2 * m] = f2_fma(k[0], vc[c], f2_mul(S[c][2 * m], g[0]));
        S[c][2 * m + 1] = f2_fma(k[1], vc[c], f2_mul(S[c][2 * m + 1], g[1]));
        o[c] = f2_fma(S[c][2 * m + 1], q[1], m == 0 ? f2_mul(S[c][0], q[0]) : f2_fma(S[c][2 * m], q[0], o[c]));
      }
    }
#pragma unroll
    for (int c = 0; c < RC; ++c) {
      const float2 p = f2_unpack(o[c]);
      r[t][c] = p.x + p.y;
    }
  }
#pragma unroll
  for (int t = 0; t < GT; ++t) {
    float* p = share + (t0 + t) * 128 * RC;
    if constexpr (RC == 4) *reinterpret_cast<float4*>(p) = make_float4(r[t][0], r[t][1], r[t][2], r[t][3]);
    else *reinterpret_cast<float2*>(p) = make_float2(r[t][0], r[t][1]);
  }
}
// read-outs of the nb tokens of one stage, times `scale` (pt: 0 .. 127).  Item = (token, group of RC columns) with KL shares; P threads share an item
// when there are fewer items than threads; every item starts at a share of its own, so that a quarter warp meets all banks.
template <typename E, int DK>
__device__ __forceinline__ void gla_read_out(const float* shares, int pt, int nb, float scale, float* out, size_t out_ld, int n_cols) {
  typedef GlaTile<E, DK> L;
  constexpr int RC = L::RC, KL = L::KL, GRP = 128 / KL, ITEMS = L::TB * GRP, P = ITEMS < 128 ? 128 / ITEMS : 1, N = KL / P;
#pragma unroll
  for (int it = pt / P; it < ITEMS; it += 128 / P) {
    const int tt = it / GRP, g = it % GRP;
    const float* p = shares + ((size_t)tt * 128 + g * KL + (pt % P) * N) * RC;
    float s[RC];
#pragma unroll
    for (int c = 0; c < RC; ++c) s[c] = 0.f;
    if (tt < nb) {
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const float* x = p + ((i + it) % N) * RC;
        if constexpr (RC == 4) {
          const float4 v = *reinterpret_cast<const float4*>(x);
          s[0] += v.x, s[1] += v.y, s[2] += v.z, s[3] += v.w;
        } else {
          const float2 v = *reinterpret_cast<const float2*>(x);
          s[0] += v.x, s[1] += v.y;
        }
      }
    }
#pragma unroll
    for (int c = 0; c < RC; ++c) {
#pragma unroll
      for (int d = 1; d < P; d <<= 1) s[c] += __shfl_xor_sync(0xffffffffu, s[c], d);
      if (tt < nb && pt % P == 0 && g * RC + c < n_cols) out[(size_t)tt * out_ld + g * RC + c] = s[c] * scale;
    }
  }
}

template <typename E, int DK>
__global__ void __launch_bounds__(256) gla_seq_kernel(GlaArgs a) {
  typedef GlaTile<E, DK> L;
  constexpr int TB = L::TB, COLS = L::COLS, RK = L::RK, RC = L::RC, KL = L::KL, NS = L::kStages;
  extern __shared__ __align__(16) unsigned char gla_sm[];
  float* const shares = reinterpret_cast<float*>(gla_sm + (size_t)NS * L::kStage);
  const int e = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, dim = a.dim, vdim = a.vdim, col0 = blockIdx.z * COLS;
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int n = a.len[e], r0 = a.row0[e], n_stages = (n + TB - 1) / TB;
  const size_t out_ld = (size_t)a.H * vdim;
  if (tid >= 128) {
    const int pt = tid - 128;
    const E* X = static_cast<const E*>(a.qkv) + (size_t)r0 * a.ld;
    const float* Z = a.zc + (size_t)r0 * a.ld_zc + h * dim;
    const int qo = a.q_off + h * dim, ko = a.k_off + h * dim, vo = a.v_off + h * vdim + col0;
    constexpr int EP = 16 / sizeof(E), VP = COLS < EP ? COLS : EP;  // entries of a 16-byte piece; of a piece of v
    // whole pieces of every row start on 16-byte boundaries (and heads end with a whole piece)
    const bool rows_ok = ((a.ld | qo | ko | dim) % EP) == 0 && (reinterpret_cast<uintptr_t>(X) & 15) == 0;
    const bool v_ok = ((a.ld | vo | vdim) % EP) == 0 && (reinterpret_cast<uintptr_t>(X) & 15) == 0 && COLS % EP == 0;
    const bool z_ok = ((a.ld_zc | (h * dim) | dim) % 4) == 0 && (reinterpret_cast<uintptr_t>(Z) & 15) == 0;
    auto load = [&](int b) {
      unsigned char* st = gla_sm + (size_t)(b % NS) * L::kStage;
      E* ks = reinterpret_cast<E*>(st);
      E* qs = reinterpret_cast<E*>(st + L::kQ);
      E* vs = reinterpret_cast<E*>(st + L::kV);
      float* gs = reinterpret_cast<float*>(st + L::kG);
      const int t0 = b * TB, nb = min(TB, n - t0);
      if (rows_ok) {
#pragma unroll
        for (int i = pt; i < TB * (DK / EP); i += 128) {
          const int tt = i / (DK / EP), d = (i % (DK / EP)) * EP;
          if (tt < nb && d < dim) {
            const E* row = X + (size_t)(t0 + tt) * a.ld;
            cp_async16(ks + tt * DK + d, row + ko + d);
            cp_async16(qs + tt * DK + d, row + qo + d);
          }
        }
      } else {
        for (int i = pt; i < nb * dim; i += 128) {
          const int tt = i / dim, d = i % dim;
          const E* row = X + (size_t)(t0 + tt) * a.ld;
          ks[tt * DK + d] = row[ko + d];
          qs[tt * DK + d] = row[qo + d];
        }
      }
      if (v_ok) {
#pragma unroll
        for (int i = pt; i < TB * (COLS / VP); i += 128) {
          const int tt = i / (COLS / VP), c = (i % (COLS / VP)) * VP;
          if (tt < nb && col0 + c < vdim) cp_async16(vs + tt * COLS + c, X + (size_t)(t0 + tt) * a.ld + vo + c);
        }
      } else {
        for (int i = pt; i < nb * COLS; i += 128) {
          const int tt = i / COLS, c = i % COLS;
          if (col0 + c < vdim) vs[tt * COLS + c] = X[(size_t)(t0 + tt) * a.ld + vo + c];
        }
      }
      if (z_ok) {
#pragma unroll
        for (int i = pt; i < TB * (DK / 4); i += 128) {
          const int tt = i / (DK / 4), d = (i % (DK / 4)) * 4;
          if (tt < nb && d < dim) cp_async16(gs + tt * DK + d, Z + (size_t)(t0 + tt) * a.ld_zc + d);
        }
      } else {
        for (int i = pt; i < nb * DK; i += 128) {
          const int tt = i / DK, d = i % DK;
          if (d < dim) gs[tt * DK + d] = Z[(size_t)(t0 + tt) * a.ld_zc + d];
        }
      }
    };
    // pre-activations -> decays in place: every thread turns the four-entry pieces that it brought itself
    auto decays = [&](int b) {
      float* gs = reinterpret_cast<float*>(gla_sm + (size_t)(b % NS) * L::kStage + L::kG);
      const int nb = min(TB, n - b * TB);
      if (z_ok) {
        for (int i = pt; i < nb * (DK / 4); i += 128) {
          const int tt = i / (DK / 4), d = (i % (DK / 4)) * 4;
          if (d >= dim) continue;
#pragma unroll
          for (int u = 0; u < 4; ++u) gs[tt * DK + d + u] = logistic_decay(gs[tt * DK + d + u] + a.bias[h * dim + d + u], a.inv_tau);
        }
      } else {
        for (int i = pt; i < nb * DK; i += 128) {
          const int tt = i / DK, d = i % DK;
          if (d < dim) gs[tt * DK + d] = logistic_decay(gs[tt * DK + d] + a.bias[h * dim + d], a.inv_tau);
        }
      }
    };
    const float qscale = 1.f / sqrtf((float)dim);
    auto read_out = [&](int b) {
      gla_read_out<E, DK>(shares + (b & 1) * L::kShares, pt, min(TB, n - b * TB), qscale, a.out + (size_t)(r0 + b * TB) * out_ld + h * vdim + col0, out_ld,
                          vdim - col0);
    };
    if (dim < DK || col0 + COLS > vdim) {  // what no copy writes stays zero: padded key entries and columns contribute nothing
      for (int i = pt * 16; i < NS * L::kStage; i += 128 * 16) *reinterpret_cast<uint4*>(gla_sm + i) = make_uint4(0, 0, 0, 0);
      asm volatile("bar.sync 1, 128;" ::: "memory");
    }
#pragma unroll
    for (int b = 0; b < NS - 1; ++b) {
      if (b < n_stages) load(b);
      cp_async_commit();
    }
    for (int b = 0; b < n_stages; ++b) {
      asm volatile("cp.async.wait_group %0;" ::"n"(NS - 2) : "memory");
      if (!a.ready) decays(b);
      __syncthreads();  // stage b has landed; the recurrence is done with the stage before it, whose place the next load takes
      if (b + NS - 1 < n_stages) load(b + NS - 1);
      cp_async_commit();
      if (b > 0) read_out(b - 1);
    }
    __syncthreads();  // the last stage's shares are complete
    read_out(n_stages - 1);
    return;
  }
  // ---- recurrence
  const int ksl = tid % KL, cl = RC * (tid / KL), n_cols = vdim - col0 - cl;  // columns of this thread inside the head (may be none)
  float* S_g = a.state + (size_t)a.slot[e] * a.slot_stride + (size_t)h * dim * vdim + col0 + cl;  // [dim][vdim]
  auto key = [&](int j) { return ((j >> 1) * KL + ksl) * 4 + (j & 1) * 2; };                      // first key entry of pair j
  F2 S[RC][RK / 2];
#pragma unroll
  for (int j = 0; j < RK / 2; ++j)
#pragma unroll
    for (int c = 0; c < RC; ++c) {
      const int i = key(j);
      S[c][j] = f2_pack(c < n_cols && i < dim ? S_g[(size_t)i * vdim + c] : 0.f, c < n_cols && i + 1 < dim ? S_g[(size_t)(i + 1) * vdim + c] : 0.f);
    }
  for (int b = 0; b < n_stages; ++b) {
    __syncthreads();
    const unsigned char* sm = gla_sm + (size_t)(b % NS) * L::kStage;
    float* share = shares + (b & 1) * L::kShares + tid * RC;
    const int nb = min(TB, n - b * TB);
    int tt = 0;
    for (; tt + kGlaGroup <= nb; tt += kGlaGroup) gla_tokens<E, DK, kGlaGroup>(S, sm, share, tt, ksl, cl);
    for (; tt < nb; ++tt) gla_tokens<E, DK, 1>(S, sm, share, tt, ksl, cl);
  }
  __syncthreads();  // the last stage's shares are complete
#pragma unroll
  for (int j = 0; j < RK / 2; ++j)
#pragma unroll
    for (int c = 0; c < RC; ++c) {
      const int i = key(j);
      const float2 w = f2_unpack(S[c][j]);
      if (c < n_cols && i < dim) S_g[(size_t)i * vdim + c] = w.x;
      if (c < n_cols && i + 1 < dim) S_g[(size_t)(i + 1) * vdim + c] = w.y;
    }
}

template <typename E, int DK>
static void launch_gla_t(const GlaArgs& a, int entries, cudaStream_t st) {
  constexpr size_t need = GlaTile<E, DK>::kSmem, apart = 116 * 1024, most = need > apart ? need : apart;
  static_assert(most <= 227 * 1024, "stages exceed shared memory");
  const dim3 g(entries, a.H, (a.vdim + GlaTile<E, DK>::COLS - 1) / GlaTile<E, DK>::COLS);
  static bool attr_set = false;  // per template instance
  if (!attr_set) {
    cudaFuncSetAttribute(gla_seq_kernel<E, DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most);
    attr_set = true;
  }
  // as for the delta rule: two CTAs never share an SM while there is one for each
  launch(gla_seq_kernel<E, DK>, g, dim3(256), (long)g.x * g.y * g.z <= sm_count() ? most : need, st, true, a);
}
template <typename E>
static int launch_gla(const GlaArgs& a, int entries, cudaStream_t st) {
  if (a.dim > 256) return -2;
  if (a.dim <= 32) launch_gla_t<E, 32>(a, entries, st);
  else if (a.dim <= 64) launch_gla_t<E, 64>(a, entries, st);
  else if (a.dim <= 128) launch_gla_t<E, 128>(a, entries, st);
  else launch_gla_t<E, 256>(a, entries, st);
  return (int)cudaGetLastError();
}

// z <- logistic(z + bias)^inv_tau in place, C entries per token
__global__ void logistic_decay_kernel(float* __restrict__ z, const float* __restrict__ bias, float inv_tau, long total, int C) {
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x)
    z[i] = logistic_decay(z[i] + bias[i % C], inv_tau);
}

// z <- exp(-exp(a_log[head]) * softplus(z + dt_bias)) in place, C = heads * dim entries per token
__global__ void channel_decay_kernel(float* __restrict__ z, const float* __restrict__ a_log, const float* __restrict__ dt_bias, long total, int C, int dim) {
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
    const int c = (int)(i % C);
    z[i] = expf(-expf(a_log[c / dim]) * softplusf_(z[i] + dt_bias[c]));
  }
}

// out[t, h, j] = E( (o[t,h,j] / den[t,h]) / sqrt(mean_j(.^2) + eps) * w[h * w_stride + j] * act(gate[t, gate_off + h*vdim + j]) )
// times `factor`, rows of stride ld_out.  act 0: silu, 1: logistic.  act 2: the silu gate comes BEFORE the norm, out = rms_norm(o * silu(gate)) * w.  den may be null.
// One warp per (token, head); "head" may be any equal part of the row (norm groups).
template <typename E>
__global__ void head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ den, const E* __restrict__ w, int w_stride,
                                      const E* __restrict__ gate, int ld_gate, int gate_off, E* __restrict__ out, int ld_out, float factor, int H, int vdim,
                                      float eps, int act, long pairs) {
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int lane = threadIdx.x & 31;
  const long pr = (long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (pr >= pairs) return;
  const long t = pr / H;
  const int h = (int)(pr % H);
  const float* orow = o + pr * vdim;
  float ss = 0.f;
  for (int j = lane; j < vdim; j += 32) {
    float v = den ? orow[j] / den[pr] : orow[j];
    if (act == 2) {
      const float gz = to_f(gate[(size_t)t * ld_gate + gate_off + h * vdim + j]);
      v *= gz / (1.f + expf(-gz));
    }
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)vdim + eps);
  for (int j = lane; j < vdim; j += 32) {
    const float v = den ? orow[j] / den[pr] : orow[j];
    const float gz = to_f(gate[(size_t)t * ld_gate + gate_off + h * vdim + j]);
    const float ga = act == 1 ? 1.f / (1.f + expf(-gz)) : gz / (1.f + expf(-gz));
    out[(size_t)t * ld_out + h * vdim + j] =
        from_f<E>(factor * (act == 2 ? (v * ga) * inv * to_f(w[(size_t)h * w_stride + j]) : v * inv * to_f(w[(size_t)h * w_stride + j]) * ga));
  }
}

// the same for few (token, head) pairs of many entries each (a decode step with wide norm groups): one CTA per pair
template <typename E>
__global__ void head_norm_gate_wide_kernel(const float* __restrict__ o, const float* __restrict__ den, const E* __restrict__ w, int w_stride,
                                           const E* __restrict__ gate, int ld_gate, int gate_off, E* __restrict__ out, int ld_out, float factor, int H,
                                           int vdim, float eps, int act) {
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const long pr = blockIdx.x, t = pr / H;
  const int h = (int)(pr % H);
  const float* orow = o + pr * vdim;
  const float dn = den ? den[pr] : 1.f;
  float v[4], ga[4];  // up to 4 entries per thread (vdim <= 4 * blockDim.x)
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    const int j = threadIdx.x + u * blockDim.x;
    v[u] = 0.f;
    ga[u] = 0.f;
    if (j < vdim) {
      const float gz = to_f(gate[(size_t)t * ld_gate + gate_off + h * vdim + j]);
      ga[u] = act == 1 ? 1.f / (1.f + expf(-gz)) : gz / (1.f + expf(-gz));
      v[u] = den ? orow[j] / dn : orow[j];
      if (act == 2) v[u] *= ga[u];
      ss = fmaf(v[u], v[u], ss);
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)vdim + eps);
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    const int j = threadIdx.x + u * blockDim.x;
    if (j < vdim)
      out[(size_t)t * ld_out + h * vdim + j] =
          from_f<E>(factor * (act == 2 ? v[u] * inv * to_f(w[(size_t)h * w_stride + j]) : v[u] * inv * to_f(w[(size_t)h * w_stride + j]) * ga[u]));
  }
}

// ---- real-gated linear recurrent unit.  z holds the gates' pre-activations without bias: block b of n channels has r at b * 2n + j and i
// at b * 2n + n + j.  out = E(S * gelu(y + y_bias)), gelu in its tanh form.
struct LruArgs {
  const void *u, *y, *y_bias;  // [tokens, ld_u] convolved input, [tokens, ld_y] raw branch, its bias [C] or null
  const float *z, *r_bias, *i_bias, *lam;
  float* state;                // [C] per slot
  const int *slot, *row0, *len;
  void* out;
  long slot_stride;
  int ld_u, ld_y, ldz, ld_out, C, n;  // n: channels of a gate block
  float rate;
};
__device__ __forceinline__ float gelu_tanh_(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));  // sqrt(2 / pi)
}
// the affine map S -> a S + b of one token
__device__ __forceinline__ float2 lru_map(float u, float zr, float zi, float neg_rate) {
  const float la = neg_rate * sigmoidf_(zr);
  return make_float2(expf(la), sqrtf(fmaxf(-expm1f(2.f * la), 0.f)) * sigmoidf_(zi) * u);  // 1 - a^2 = -(e^(2 log a) - 1)
}

// few tokens per entry: one thread per channel, token by token
template <typename E>
__global__ void lru_step_kernel(LruArgs a) {
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int c = blockIdx.x * blockDim.x + threadIdx.x, e = blockIdx.y;
  if (c >= a.C) return;
  const int n = a.len[e], r0 = a.row0[e], zo = (c / a.n) * 2 * a.n + c % a.n;
  float* st = a.state + (size_t)a.slot[e] * a.slot_stride + c;
  const float rb = a.r_bias[c], ib = a.i_bias[c], neg = -a.rate * softplusf_(a.lam[c]), yb = a.y_bias ? to_f(static_cast<const E*>(a.y_bias)[c]) : 0.f;
  float S = st[0];
#pragma unroll 2
  for (int o = 0; o < n; ++o) {
    const size_t t = (size_t)(r0 + o);
    const float2 m = lru_map(to_f(static_cast<const E*>(a.u)[t * a.ld_u + c]), a.z[t * a.ldz + zo] + rb, a.z[t * a.ldz + zo + a.n] + ib, neg);
    S = fmaf(m.x, S, m.y);
    static_cast<E*>(a.out)[t * a.ld_out + c] = from_f<E>(S * gelu_tanh_(to_f(static_cast<const E*>(a.y)[t * a.ld_y + c]) + yb));
  }
  st[0] = S;
}

// a prompt portion: CTA = 16 channels of one entry, 32 groups of TPT consecutive tokens at a time.  Every thread composes the maps of its
// tokens, one warp per channel scans the 32 composed maps with shuffles, and every thread then runs its tokens from its start state.
template <typename E, int TPT>
__global__ void __launch_bounds__(512) lru_scan_kernel(LruArgs a) {
  constexpr int CH = 16, NG = 32;
  __shared__ float sa[NG][CH + 1], sb[NG][CH + 1], s_in[NG][CH + 1], carry[CH];
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int tid = threadIdx.x, ch = tid % CH, tg = tid / CH, c = blockIdx.x * CH + ch, e = blockIdx.y, lane = tid & 31, warp = tid >> 5;
  const bool on = c < a.C;
  const int n = a.len[e], r0 = a.row0[e], zo = on ? (c / a.n) * 2 * a.n + c % a.n : 0;
  float* st = a.state + (size_t)a.slot[e] * a.slot_stride;
  float rb = 0.f, ib = 0.f, neg = 0.f, yb = 0.f;
  if (on) {
    rb = a.r_bias[c];
    ib = a.i_bias[c];
    neg = -a.rate * softplusf_(a.lam[c]);
    yb = a.y_bias ? to_f(static_cast<const E*>(a.y_bias)[c]) : 0.f;
  }
  if (tid < CH) carry[tid] = blockIdx.x * CH + tid < a.C ? st[blockIdx.x * CH + tid] : 0.f;
  for (int b0 = 0; b0 < n; b0 += NG * TPT) {
    float2 m[TPT];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int k = 0; k < TPT; ++k) {
      const int o = b0 + tg * TPT + k;
      m[k] = make_float2(1.f, 0.f);
      if (on && o < n) {
        const size_t t = (size_t)(r0 + o);
        m[k] = lru_map(to_f(static_cast<const E*>(a.u)[t * a.ld_u + c]), a.z[t * a.ldz + zo] + rb, a.z[t * a.ldz + zo + a.n] + ib, neg);
      }
      A *= m[k].x;
      B = fmaf(m[k].x, B, m[k].y);
    }
    sa[tg][ch] = A;
    sb[tg][ch] = B;
    __syncthreads();
    {  // warp w: channel w, lane = token group; inclusive scan of the composed maps
      float xa = sa[lane][warp], xb = sb[lane][warp];
#pragma unroll
      for (int d = 1; d < NG; d <<= 1) {
        const float pa = __shfl_up_sync(0xffffffffu, xa, d), pb = __shfl_up_sync(0xffffffffu, xb, d);
        if (lane >= d) {
          xb = fmaf(xa, pb, xb);
          xa *= pa;
        }
      }
      const float s0 = carry[warp];
      float ea = __shfl_up_sync(0xffffffffu, xa, 1), eb = __shfl_up_sync(0xffffffffu, xb, 1);
      if (lane == 0) ea = 1.f, eb = 0.f;
      s_in[lane][warp] = fmaf(ea, s0, eb);
      __syncwarp();  // every lane has read the old carry
      if (lane == NG - 1) carry[warp] = fmaf(xa, s0, xb);
    }
    __syncthreads();
    float S = s_in[tg][ch];
#pragma unroll
    for (int k = 0; k < TPT; ++k) {
      const int o = b0 + tg * TPT + k;
      S = fmaf(m[k].x, S, m[k].y);
      if (on && o < n) {
        const size_t t = (size_t)(r0 + o);
        static_cast<E*>(a.out)[t * a.ld_out + c] = from_f<E>(S * gelu_tanh_(to_f(static_cast<const E*>(a.y)[t * a.ld_y + c]) + yb));
      }
    }
  }
  __syncthreads();
  if (tid < CH && blockIdx.x * CH + tid < a.C) st[blockIdx.x * CH + tid] = carry[tid];
}

template <typename E, int MODE>
static int launch_seq(const SeqArgs& a, int entries, cudaStream_t st) {
  if (a.dim > 256) return -2;
  const int dk = a.dim <= 32 ? 32 : a.dim <= 64 ? 64 : a.dim <= 128 ? 128 : 256;
  const int cols = 128 / (dk / 16);
  const dim3 grid(entries, a.H, (a.vdim + cols - 1) / cols), block(MODE == 1 ? 160 : 128);
  if (dk == 32) launch(recurrent_seq_kernel<E, 32, MODE>, grid, block, 0, st, true, a);
  else if (dk == 64) launch(recurrent_seq_kernel<E, 64, MODE>, grid, block, 0, st, true, a);
  else if (dk == 128) launch(recurrent_seq_kernel<E, 128, MODE>, grid, block, 0, st, true, a);
  else launch(recurrent_seq_kernel<E, 256, MODE>, grid, block, 0, st, true, a);
  return (int)cudaGetLastError();
}

}  // namespace pk

using namespace pk;

extern "C" int pk_causal_conv_silu(const void* in, int ld_in, const void* w, float* state, long slot_stride, const int* req, const int* slot,
                                   const int* row0, const int* len, void* out, int ld_out, int channels, int taps, int tokens, int entries, int f32,
                                   pk_stream st) {
  return pk_causal_conv_silu_bias(in, ld_in, w, nullptr, state, slot_stride, req, slot, row0, len, out, ld_out, channels, taps, tokens, entries, f32, st);
}

extern "C" int pk_causal_conv_silu_bias(const void* in, int ld_in, const void* w, const void* bias, float* state, long slot_stride, const int* req,
                                        const int* slot, const int* row0, const int* len, void* out, int ld_out, int channels, int taps, int tokens,
                                        int entries, int f32, pk_stream st) {
  if (!req) return -1;
  return pk_causal_conv(in, ld_in, nullptr, w, bias, 1, state, slot_stride, slot, row0, len, out, ld_out, channels, taps, tokens, entries, f32, st);
}

extern "C" int pk_causal_conv(const void* in, int ld_in, const void* in_bias, const void* w, const void* bias, int act, float* state, long slot_stride,
                              const int* slot, const int* row0, const int* len, void* out, int ld_out, int channels, int taps, int tokens, int entries,
                              int f32, pk_stream st) {
  if (!in || !w || !state || !slot || !row0 || !len || !out || channels <= 0 || taps <= 0 || tokens <= 0 || entries <= 0 || act < 0 || act > 1) return -1;
  const int gs = std::max(8, taps - 1);  // tokens per group; an entry has at most one ragged group
  const int threads = channels >= 128 * 148 || tokens > 256 ? 128 : 64;
  const dim3 g((channels + threads - 1) / threads, tokens / gs + entries);
  if (g.y > 65535) return -2;
#define PK_CONV(E, TAPS)                                                                                                                      \
  launch(causal_conv_kernel<E, TAPS>, g, dim3(threads), 0, st, true, (const E*)in, ld_in, (const E*)in_bias, (const E*)w, (const E*)bias, state, \
         slot_stride, slot, row0, len, (E*)out, ld_out, channels, taps, act, entries, gs)
  if (f32) {
    if (taps == 4) PK_CONV(float, 4);
    else PK_CONV(float, 0);
  } else {
    if (taps == 4) PK_CONV(bf16, 4);
    else PK_CONV(bf16, 0);
  }
#undef PK_CONV
  return (int)cudaGetLastError();
}

static bool seq_args_ok(const void* qkv, const float* z, const float* p0, const float* p1, float* state, const int* slot, const int* row0, const int* len,
                        float* out, int H, int G, int dim, int vdim, int entries) {
  return qkv && z && p0 && p1 && state && slot && row0 && len && out && H > 0 && G > 0 && H % G == 0 && dim > 0 && vdim > 0 && entries > 0;
}

extern "C" int pk_gated_delta_seq(const void* qkv, int ld, int q_off, int k_off, int v_off, const float* z, int ldz, int decay_off, int beta_off,
                                  const float* a_log, const float* dt_bias, float* state, long slot_stride, const int* slot, const int* row0,
                                  const int* len, float* out, int heads, int kv_heads, int dim, int vdim, int entries, int f32, pk_stream st) {
  if (!seq_args_ok(qkv, z, a_log, dt_bias, state, slot, row0, len, out, heads, kv_heads, dim, vdim, entries)) return -1;
  SeqArgs a{qkv, ld, q_off, k_off, v_off, z, ldz, decay_off, beta_off, a_log, dt_bias, state, slot_stride, slot, row0, len, out, nullptr,
            heads, kv_heads, dim, vdim, 0.f};
  return f32 ? launch_delta<float, false>(a, entries, st) : launch_delta<bf16, false>(a, entries, st);
}

extern "C" int pk_channel_delta_seq(const void* qkv, int ld, int q_off, int k_off, int v_off, const float* z, int ldz, int beta_off, const float* decay,
                                    int ld_decay, int decay_ready, const float* a_log, const float* dt_bias, float* state, long slot_stride, const int* slot,
                                    const int* row0, const int* len, float* out, int heads, int kv_heads, int dim, int vdim, int entries, int f32,
                                    pk_stream st) {
  if (!seq_args_ok(qkv, z, a_log, dt_bias, state, slot, row0, len, out, heads, kv_heads, dim, vdim, entries) || !decay || ld_decay < heads * dim) return -1;
  SeqArgs a{qkv, ld, q_off, k_off, v_off, z, ldz, 0, beta_off, a_log, dt_bias, state, slot_stride, slot, row0, len, out, nullptr,
            heads, kv_heads, dim, vdim, 0.f, nullptr, 0, 0, nullptr, decay, ld_decay, decay_ready};
  return f32 ? launch_delta<float, true>(a, entries, st) : launch_delta<bf16, true>(a, entries, st);
}

extern "C" int pk_mlstm_seq(const void* qkv, int ld, int q_off, int k_off, int v_off, const float* z, int ldz, int forget_off, int input_off,
                            const float* input_bias, const float* forget_bias, float cap, float* state, long slot_stride, const int* slot,
                            const int* row0, const int* len, float* out, float* den, int heads, int dim, int vdim, int entries, int f32,
                            pk_stream st) {
  if (!seq_args_ok(qkv, z, input_bias, forget_bias, state, slot, row0, len, out, heads, heads, dim, vdim, entries) || !den || !(cap > 0.f)) return -1;
  SeqArgs a{qkv, ld, q_off, k_off, v_off, z, ldz, forget_off, input_off, input_bias, forget_bias, state, slot_stride, slot, row0, len, out, den,
            heads, heads, dim, vdim, cap};
  return f32 ? launch_seq<float, 1>(a, entries, st) : launch_seq<bf16, 1>(a, entries, st);
}

extern "C" int pk_head_norm_gate(const float* o, const float* den, const void* w, int w_stride, const void* gate, int ld_gate, int gate_off, void* out,
                                 int tokens, int heads, int vdim, float eps, int act, int f32, pk_stream st) {
  return pk_head_norm_gate_ex(o, den, w, w_stride, gate, ld_gate, gate_off, out, heads * vdim, 1.f, tokens, heads, vdim, eps, act, f32, st);
}

extern "C" int pk_head_norm_gate_ex(const float* o, const float* den, const void* w, int w_stride, const void* gate, int ld_gate, int gate_off, void* out,
                                    int ld_out, float factor, int tokens, int heads, int vdim, float eps, int act, int f32, pk_stream st) {
  if (!o || !w || !gate || !out || tokens <= 0 || heads <= 0 || vdim <= 0 || ld_out < heads * vdim || act < 0 || act > 2) return -1;
  const long pairs = (long)tokens * heads;
  if (vdim >= 256 && vdim <= 4096 && pairs <= 1024) {  // few wide pairs: a CTA each, so that a decode step is not one warp's loop
    const dim3 gw((unsigned)pairs), bw(vdim <= 512 ? 128 : vdim <= 1024 ? 256 : 1024);
    if (f32)
      launch(head_norm_gate_wide_kernel<float>, gw, bw, 0, st, true, o, den, (const float*)w, w_stride, (const float*)gate, ld_gate, gate_off, (float*)out,
             ld_out, factor, heads, vdim, eps, act);
    else
      launch(head_norm_gate_wide_kernel<bf16>, gw, bw, 0, st, true, o, den, (const bf16*)w, w_stride, (const bf16*)gate, ld_gate, gate_off, (bf16*)out,
             ld_out, factor, heads, vdim, eps, act);
    return (int)cudaGetLastError();
  }
  const dim3 g((unsigned)((pairs + 3) / 4));
  if (f32)
    launch(head_norm_gate_kernel<float>, g, dim3(128), 0, st, true, o, den, (const float*)w, w_stride, (const float*)gate, ld_gate, gate_off, (float*)out,
           ld_out, factor, heads, vdim, eps, act, pairs);
  else
    launch(head_norm_gate_kernel<bf16>, g, dim3(128), 0, st, true, o, den, (const bf16*)w, w_stride, (const bf16*)gate, ld_gate, gate_off, (bf16*)out, ld_out,
           factor, heads, vdim, eps, act, pairs);
  return (int)cudaGetLastError();
}

extern "C" int pk_ssd_seq(const void* xbc, int ld, int x_off, int b_off, int c_off, const void* dt, int ld_dt, int dt_off, const float* a_log,
                          const float* dt_bias, const float* d_skip, float* state, long slot_stride, const int* slot, const int* row0, const int* len,
                          float* out, int heads, int groups, int state_dim, int vdim, int entries, int f32, pk_stream st) {
  if (!xbc || !dt || !a_log || !dt_bias || !d_skip || !state || !slot || !row0 || !len || !out || heads <= 0 || groups <= 0 || heads % groups ||
      state_dim <= 0 || vdim <= 0 || entries <= 0)
    return -1;
  SeqArgs a{xbc, ld, c_off, b_off, x_off, nullptr, 0, 0, 0, a_log, dt_bias, state, slot_stride, slot, row0, len, out, nullptr,
            heads, groups, state_dim, vdim, 0.f, dt, ld_dt, dt_off, d_skip};
  return f32 ? launch_seq<float, 2>(a, entries, st) : launch_seq<bf16, 2>(a, entries, st);
}

extern "C" int pk_lru_seq(const void* u, int ld_u, const float* z, int ldz, const float* r_bias, const float* i_bias, const float* lam, float rate,
                          int blocks, const void* y, int ld_y, const void* y_bias, float* state, long slot_stride, const int* slot, const int* row0,
                          const int* len, void* out, int ld_out, int channels, int tokens, int entries, int f32, pk_stream st) {
  if (!u || !z || !r_bias || !i_bias || !lam || !y || !state || !slot || !row0 || !len || !out || channels <= 0 || blocks <= 0 || channels % blocks ||
      tokens <= 0 || entries <= 0 || !(rate > 0.f))
    return -1;
  LruArgs a{u, y, y_bias, z, r_bias, i_bias, lam, state, slot, row0, len, out, slot_stride, ld_u, ld_y, ldz, ld_out, channels, channels / blocks, rate};
  if (tokens <= 8 * entries) {
    const dim3 g((channels + 63) / 64, entries);
    if (f32) launch(lru_step_kernel<float>, g, dim3(64), 0, st, true, a);
    else launch(lru_step_kernel<bf16>, g, dim3(64), 0, st, true, a);
  } else {
    const dim3 g((channels + 15) / 16, entries);
    if (f32) launch(lru_scan_kernel<float, 8>, g, dim3(512), 0, st, true, a);
    else launch(lru_scan_kernel<bf16, 8>, g, dim3(512), 0, st, true, a);
  }
  return (int)cudaGetLastError();
}

extern "C" int pk_channel_decay(float* z, const float* a_log, const float* dt_bias, int tokens, int heads, int dim, pk_stream st) {
  if (!z || !a_log || !dt_bias || tokens <= 0 || heads <= 0 || dim <= 0) return -1;
  const long total = (long)tokens * heads * dim;
  launch(channel_decay_kernel, dim3((unsigned)std::min<long>((total + 255) / 256, 148L * 8)), dim3(256), 0, st, true, z, a_log, dt_bias, total, heads * dim, dim);
  return (int)cudaGetLastError();
}

extern "C" int pk_gla_seq(const void* qkv, int ld, int q_off, int k_off, int v_off, const float* decay, int ld_decay, int decay_ready, const float* bias,
                          float tau, float* state, long slot_stride, const int* slot, const int* row0, const int* len, float* out, int heads, int dim,
                          int vdim, int entries, int f32, pk_stream st) {
  if (!qkv || !decay || !bias || !state || !slot || !row0 || !len || !out || heads <= 0 || dim <= 0 || vdim <= 0 || entries <= 0 ||
      ld_decay < heads * dim || !(tau > 0.f))
    return -1;
  GlaArgs a{qkv, ld, q_off, k_off, v_off, decay, ld_decay, decay_ready, bias, 1.f / tau, state, slot_stride, slot, row0, len, out, heads, dim, vdim};
  return f32 ? launch_gla<float>(a, entries, st) : launch_gla<bf16>(a, entries, st);
}

extern "C" int pk_logistic_decay(float* z, const float* bias, float tau, int tokens, int channels, pk_stream st) {
  if (!z || !bias || tokens <= 0 || channels <= 0 || !(tau > 0.f)) return -1;
  const long total = (long)tokens * channels;
  launch(logistic_decay_kernel, dim3((unsigned)std::min<long>((total + 255) / 256, 148L * 8)), dim3(256), 0, st, true, z, bias, 1.f / tau, total, channels);
  return (int)cudaGetLastError();
}
