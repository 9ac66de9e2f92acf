// Grouped-query attention whose heads' scores are mixed and whose weights are logistic, over the paged K/V cache of gqa_attention.cu:
//   s_h(j)  = scale * q_h . k_j(head h / (H / G))
//   z_h(j)  = sum_g mix[h][g] s_g(j) + bias[h]              (mix [H, H] may be absent: z_h = s_h + bias[h])
//   out_h   = out_scale * logistic(gate_h) * sum over visible j of logistic(z_h(j)) v_j        (gate may be absent)
// Weights are not normalised over keys, so a row's result is a plain sum over keys: there is no running maximum, and partial sums over
// any split of the key axis simply add up.  Scores, mixing, weights and sums are fp32; the element type E (bf16 or float) is that of the
// activations and of the cache.  The mixing couples all heads, so a CTA always works on every head of its rows.
//   mixed_attention_kernel       one CTA per (query row, share of the keys), any sizes, both element types: keys in blocks through shared
//                                memory, one thread per (head, key) score.  The fp32 path and odd sizes.
//   mixed_attention_mma_kernel   bf16 on the tensor cores: 16 query rows of every head per CTA (decode steps: one row), and a share of the keys.
//   mixed_attention_merge_kernel, mixed_attention_merge4_kernel   add the shares' partial sums and apply the gate.
#include <algorithm>
#include <type_traits>

#include "common.cuh"
#include "mma.cuh"
#include "typed.cuh"

namespace pk {

struct MixedArgs {
  const void *q, *cache;                       // q [tokens, H * dim]; cache as in gqa_attention.cu
  const void* mix;                             // E [H, H] or null
  const float* bias;                           // [H] or null
  const float* gate;                           // fp32 pre-activations, rows of stride gate_ld, or null
  const int *pos, *req, *page_off, *pages;
  void* out;                                   // E, rows of stride out_ld
  float* part;                                 // [splits][T][H * vdim] when the key axis is split
  long page_stride;
  int gate_ld, out_ld, page_size, T, H, G, dim, vdim, splits, tile_rows;  // tile_rows: rows of a tensor-core CTA that are in use (16, or 1 for decode steps)
  float scale, out_scale;
};

__device__ __forceinline__ float logistic_exact(float z) { return 1.f / (1.f + expf(-z)); }

// out (or the partial sum of this share) of entry i = h * vdim + d of row t
template <typename E>
__device__ __forceinline__ void mixed_store(const MixedArgs& a, int split, int t, int i, float v) {
  if (a.splits > 1) {
    a.part[((size_t)split * a.T + t) * a.H * a.vdim + i] = v;
  } else {
    const float f = a.gate ? a.out_scale * logistic_exact(a.gate[(size_t)t * a.gate_ld + i / a.vdim]) : a.out_scale;
    static_cast<E*>(a.out)[(size_t)t * a.out_ld + i] = from_f<E>(v * f);
  }
}

// shared memory of the generic kernel: q [H * dim] | K block [kb][G * dim + 1] | scores [H][kb] | weights [H][kb] | mix [H * H] | sums [H * vdim]
static inline size_t mixed_smem(int H, int G, int dim, int vdim, int kb) {
  return ((size_t)H * dim + (size_t)kb * (G * dim + 1) + 2 * (size_t)H * kb + (size_t)H * H + (size_t)H * vdim) * sizeof(float);
}

template <typename E>
__global__ void __launch_bounds__(256) mixed_attention_kernel(MixedArgs a, int kb) {
  extern __shared__ __align__(16) float mx_sm[];
  __shared__ long long off[32];  // element offset of every key of the block inside the cache
  const int H = a.H, G = a.G, dim = a.dim, vdim = a.vdim, per = H / G, ldk = G * dim + 1, tid = threadIdx.x;
  float* qs = mx_sm;
  float* ks = qs + H * dim;
  float* sc = ks + (size_t)kb * ldk;
  float* wt = sc + H * kb;
  float* mixs = wt + H * kb;
  float* acc = mixs + H * H;
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int t = blockIdx.x, split = blockIdx.y, p = a.pos[t];
  const int* pg = a.pages + a.page_off[a.req[t]];
  const E* cache = static_cast<const E*>(a.cache);
  const E* q = static_cast<const E*>(a.q) + (size_t)t * H * dim;
  for (int i = tid; i < H * dim; i += blockDim.x) qs[i] = to_f(q[i]) * a.scale;
  if (a.mix)
    for (int i = tid; i < H * H; i += blockDim.x) mixs[i] = to_f(static_cast<const E*>(a.mix)[i]);
  for (int i = tid; i < H * vdim; i += blockDim.x) acc[i] = 0.f;
  const int tok = G * (dim + vdim), n_blocks = p / kb + 1, per_split = (n_blocks + a.splits - 1) / a.splits;
  const int b_end = min(n_blocks, (split + 1) * per_split);
  for (int b = split * per_split; b < b_end; ++b) {
    const int k0 = b * kb, nk = min(kb, p + 1 - k0);
    __syncthreads();  // the previous block's readers are done
    if (tid < nk) {
      const int j = k0 + tid;
      off[tid] = (long long)pg[j / a.page_size] * a.page_stride + (long long)(j % a.page_size) * tok;
    }
    __syncthreads();
    bool staged = false;
    if constexpr (sizeof(E) == 2) {
      if (((G * dim | tok | (int)(a.page_stride & 7)) & 7) == 0 && (reinterpret_cast<uintptr_t>(cache) & 15) == 0) {
        staged = true;
        const int pr = G * dim / 8;
#pragma unroll 4
        for (int i = tid; i < nk * pr; i += blockDim.x) {
          const int kk = i / pr, c = (i % pr) * 8;
          const uint4 v = *reinterpret_cast<const uint4*>(cache + off[kk] + c);
          float* d = ks + (size_t)kk * ldk + c;
          d[0] = bf16_lo(v.x), d[1] = bf16_hi(v.x), d[2] = bf16_lo(v.y), d[3] = bf16_hi(v.y);
          d[4] = bf16_lo(v.z), d[5] = bf16_hi(v.z), d[6] = bf16_lo(v.w), d[7] = bf16_hi(v.w);
        }
      }
    }
    if (!staged)
      for (int i = tid; i < nk * G * dim; i += blockDim.x) {
        const int kk = i / (G * dim), c = i % (G * dim);
        ks[(size_t)kk * ldk + c] = to_f(cache[off[kk] + c]);
      }
    __syncthreads();
    for (int i = tid; i < H * kb; i += blockDim.x) {  // one thread per (head, key)
      const int h = i / kb, kk = i % kb;
      float s0 = 0.f, s1 = 0.f;
      if (kk < nk) {
        const float* kr = ks + (size_t)kk * ldk + (h / per) * dim;
        const float* qr = qs + h * dim;
        int d = 0;
        for (; d + 2 <= dim; d += 2) {
          s0 = fmaf(qr[d], kr[d], s0);
          s1 = fmaf(qr[d + 1], kr[d + 1], s1);
        }
        if (d < dim) s0 = fmaf(qr[d], kr[d], s0);
      }
      sc[i] = s0 + s1;
    }
    __syncthreads();
    for (int i = tid; i < H * kb; i += blockDim.x) {
      const int h = i / kb, kk = i % kb;
      float z = a.mix ? 0.f : sc[i];
      if (a.mix)
        for (int g = 0; g < H; ++g) z = fmaf(mixs[h * H + g], sc[g * kb + kk], z);
      wt[i] = kk < nk ? logistic_exact(z + (a.bias ? a.bias[h] : 0.f)) : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < H * vdim; i += blockDim.x) {  // every thread meets the sums it owns: no race
      const int h = i / vdim, d = i % vdim, c = G * dim + (h / per) * vdim + d;
      float s = acc[i];
#pragma unroll 8
      for (int kk = 0; kk < nk; ++kk) s = fmaf(wt[h * kb + kk], to_f(cache[off[kk] + c]), s);
      acc[i] = s;
    }
  }
  __syncthreads();
  for (int i = tid; i < H * vdim; i += blockDim.x) mixed_store<E>(a, split, t, i, acc[i]);
}

// ---- tensor cores (bf16).  One CTA = 16 consecutive rows of the step x every head; 32-key blocks of the request's K | V rows go through
// cp.async stages in shared memory.  Per block:
//   1. raw scores of every head, S = Q K^T (a warp owns HPW heads; heads of one group share the K fragments), to shared memory as fp32;
//   2. mixing: for a fixed row and 8 keys, [heads x heads] * [heads x 8 keys] is itself a tensor-core product.  mix is bf16 already; an
//      fp32 score enters as three bf16 terms (high, middle, low: all 24 bits), three products with fp32 accumulation.  Then bias,
//      logistic, visibility, and the weights go to shared memory as bf16;
//   3. O += P V per head, accumulators in registers.  Step 3 of a block and step 1 of the next one run without a barrier in between.
// Rows of a tile may belong to several requests: each request's keys are walked with the other rows' weights at zero.  More than 16
// heads: gridDim.z CTAs share a tile, each scoring all heads and summing 16 of them.
constexpr int kMxRows = 16, kMxKeys = 32, kMxMaxK = 4;  // kMxMaxK * 16 = most heads
constexpr int kMxLS = kMxKeys + 8;                      // floats per score row; head stride = 4 mod 16 keeps step 2's reads on distinct banks
constexpr int kMxHS = kMxRows * kMxLS + 4;
constexpr int kMxLP = kMxKeys + 8;                      // bf16 per weight row; head stride 4 mod 32 words
constexpr int kMxHP = kMxRows * kMxLP + 8;

// logistic of z from z2 = -z * log2(e), on the special-function unit (relative error of a few 2^-22; 2^z2 = inf gives 0)
__device__ __forceinline__ float fast_logistic2(float z2) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(z2));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.f));
  return r;
}
// x = hi + mid + lo exactly, each a bf16 (eight significant bits cut off at a time): the pair (x0, x1) as three packed registers
__device__ __forceinline__ uint32_t upper_halves(float x0, float x1) { return __byte_perm(__float_as_uint(x0), __float_as_uint(x1), 0x7632); }
__device__ __forceinline__ void split3(float x0, float x1, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  hi = upper_halves(x0, x1);
  const float r0 = x0 - __uint_as_float(__float_as_uint(x0) & 0xffff0000u), r1 = x1 - __uint_as_float(__float_as_uint(x1) & 0xffff0000u);
  mid = upper_halves(r0, r1);
  lo = upper_halves(r0 - __uint_as_float(__float_as_uint(r0) & 0xffff0000u), r1 - __uint_as_float(__float_as_uint(r1) & 0xffff0000u));
}

// DQ, DV: dim and vdim (EXACT: no size tests inside the unrolled products, which the compiler then schedules as one block) or their upper bounds;
// HPW: heads a warp holds; NK: at least ceil(H / 16)
// mma_bf16_16816 that the compiler may move among independent work
__device__ __forceinline__ void mma_free(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int DQ, int DV, int HPW, int NK, bool EXACT>
__global__ void __launch_bounds__(256, DQ <= 64 && HPW == 1 ? 2 : 1) mixed_attention_mma_kernel(MixedArgs a, int stages) {
  extern __shared__ __align__(16) unsigned char mm_smem[];
  __shared__ int s_req[kMxRows], s_pos[kMxRows];
  __shared__ long long s_off[2][kMxKeys];
  const int H = a.H, G = a.G, dim = EXACT ? DQ : a.dim, vdim = EXACT ? DV : a.vdim, per = H / G, tok = G * (dim + vdim), ldt = tok + 8;
  bf16* const kv0 = reinterpret_cast<bf16*>(mm_smem);                                      // [stages][keys][ldt]: K of G heads | V of G heads
  const int H16 = (H + 15) / 16 * 16;                                                         // scores of the heads H .. H16 - 1 stay zero
  float* const S = reinterpret_cast<float*>(mm_smem + (size_t)stages * kMxKeys * ldt * 2);  // [H16][kMxHS]
  bf16* const P = reinterpret_cast<bf16*>(S + (size_t)H16 * kMxHS);                          // [16][kMxHP]
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  // grid (share, tile, head slice); tiles from the end of the step first: they see the most keys
  const int t0 = (gridDim.y - 1 - blockIdx.y) * a.tile_rows, split = blockIdx.x, h_base = blockIdx.z * 16, nh = min(16, H - h_base);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5, gq = lane >> 2, tq = lane & 3;
  if (tid < kMxRows) {
    const int t = t0 + tid;
    const bool on = tid < a.tile_rows && t < a.T;
    s_req[tid] = on ? a.req[t] : -1;
    s_pos[tid] = on ? a.pos[t] : -1;
  }
  __syncthreads();
  for (int i = H * kMxHS + tid; i < H16 * kMxHS; i += blockDim.x) S[i] = 0.f;
  const bf16* q = static_cast<const bf16*>(a.q);
  const bf16* cache = static_cast<const bf16*>(a.cache);
  const int row_a = t0 + gq, row_b = t0 + gq + 8;
  const bool in_a = gq < a.tile_rows && row_a < a.T, in_b = gq + 8 < a.tile_rows && row_b < a.T;
  uint32_t qa[HPW][DQ / 16][4];
  auto load_q = [&](int i, int h) {
#pragma unroll
    for (int kk = 0; kk < DQ / 16; ++kk) {
      const int c = kk * 16 + 2 * tq;
      const bool on = h < H && kk * 16 < dim;
      const bf16* pa = q + ((size_t)row_a * H + h) * dim + c;
      const bf16* pb = q + ((size_t)row_b * H + h) * dim + c;
      qa[i][kk][0] = on && in_a ? *reinterpret_cast<const uint32_t*>(pa) : 0u;
      qa[i][kk][1] = on && in_b ? *reinterpret_cast<const uint32_t*>(pb) : 0u;
      qa[i][kk][2] = on && in_a ? *reinterpret_cast<const uint32_t*>(pa + 8) : 0u;
      qa[i][kk][3] = on && in_b ? *reinterpret_cast<const uint32_t*>(pb + 8) : 0u;
    }
  };
  const int hpb = nw * HPW;  // heads the warps hold at once
  if (H <= hpb) {
#pragma unroll
    for (int i = 0; i < HPW; ++i) load_q(i, warp * HPW + i);
  }
  // step 2's left operand: mix[h_base + row][k], rows gq and gq + 8 (the identity without a mixing matrix)
  uint32_t ta[NK][4];
  {
    auto m = [&](int h, int g) -> float {
      if (h >= H || g >= H) return 0.f;
      return a.mix ? bf2f(static_cast<const bf16*>(a.mix)[(size_t)h * H + g]) : (h == g ? 1.f : 0.f);
    };
#pragma unroll
    for (int kk = 0; kk < NK; ++kk) {
      const int g = kk * 16 + 2 * tq, h = h_base + gq;
      ta[kk][0] = pack_bf16(m(h, g), m(h, g + 1));
      ta[kk][1] = pack_bf16(m(h + 8, g), m(h + 8, g + 1));
      ta[kk][2] = pack_bf16(m(h, g + 8), m(h, g + 9));
      ta[kk][3] = pack_bf16(m(h + 8, g + 8), m(h + 8, g + 9));
    }
  }
  constexpr float kNegLog2e = -1.4426950408889634f;
  const float scale2 = a.scale * kNegLog2e;  // mixed raw score -> argument of fast_logistic2
  const float bias_a = a.bias && gq < nh ? a.bias[h_base + gq] * kNegLog2e : 0.f, bias_b = a.bias && gq + 8 < nh ? a.bias[h_base + gq + 8] * kNegLog2e : 0.f;
  float o[HPW][DV / 8][4] = {};
  // shared-memory addresses of this lane's ldmatrix rows: K fragments, V fragments (transposed), weights
  const uint32_t kv_at = smem_u32(kv0), stage_bytes = (uint32_t)(kMxKeys * ldt * 2), row16 = (uint32_t)(16 * ldt * 2);
  const uint32_t k_lane = (uint32_t)((((lane & 7) + ((lane >> 4) & 1) * 8) * ldt + ((lane >> 3) & 1) * 8) * 2);
  const uint32_t v_lane = (uint32_t)((((lane & 7) + ((lane >> 3) & 1) * 8) * ldt + ((lane >> 4) & 1) * 8 + G * dim) * 2);
  const uint32_t p_at = smem_u32(P) + (uint32_t)((((lane & 7) + ((lane >> 3) & 1) * 8) * kMxLP + ((lane >> 4) & 1) * 8) * 2);
  int r_first = 0;
  while (r_first < kMxRows && s_req[r_first] >= 0) {
    const int rq = s_req[r_first];
    int r_last = r_first;
    while (r_last + 1 < kMxRows && s_req[r_last + 1] == rq) ++r_last;
    const int p_max = s_pos[r_last], p_min = s_pos[r_first];
    const bool whole_tile = r_first == 0 && r_last == kMxRows - 1;
    const int* pg = a.pages + a.page_off[rq];
    const int n_blocks = p_max / kMxKeys + 1, per_split = (n_blocks + a.splits - 1) / a.splits;
    const int b0 = split * per_split, b_end = min(n_blocks, b0 + per_split);
    auto page_of = [&](int b) {  // page of this thread's key of block b (-1: past the last visible key)
      const int j = b * kMxKeys + tid;
      return tid < kMxKeys && j <= p_max ? pg[j / a.page_size] : -1;
    };
    auto note = [&](int b, int page) {  // cache offsets of block b's keys
      if (tid < kMxKeys) s_off[b & 1][tid] = page >= 0 ? (long long)page * a.page_stride + (long long)((b * kMxKeys + tid) % a.page_size) * tok : -1;
    };
    auto load = [&](int b) {  // K | V rows of block b into its stage
      bf16* dst = kv0 + (stages == 2 ? (b & 1) : 0) * kMxKeys * ldt;
      for (int r = warp; r < kMxKeys; r += nw) {
        const long long at = s_off[b & 1][r];
        bf16* d = dst + r * ldt;
        if (at >= 0) {
          const bf16* src = cache + at;
#pragma unroll 4
          for (int c = lane * 8; c < tok; c += 256) cp_async16(d + c, src + c);
        } else {
          for (int c = lane * 8; c < tok; c += 256) *reinterpret_cast<uint4*>(d + c) = make_uint4(0, 0, 0, 0);
        }
      }
      cp_async_commit();
    };
    // step 1 for the heads from h0 on; one_group: they read the same keys
    auto scores_of = [&](uint32_t kv, int h0, auto one_group) {
      const uint32_t k_at = kv + k_lane + (uint32_t)(h0 / per * dim * 2);
      uint32_t k_of[HPW];
#pragma unroll
      for (int i = 0; i < HPW; ++i) k_of[i] = kv + k_lane + (uint32_t)(min((h0 + i) / per, G - 1) * dim * 2);
      float* const d = S + h0 * kMxHS + gq * kMxLS + 2 * tq;
#pragma unroll
      for (int np = 0; np < kMxKeys / 16; ++np) {
        float s[HPW][2][4] = {};
#pragma unroll
        for (int kk = 0; kk < DQ / 16; ++kk) {
          if (EXACT || kk * 16 < dim) {
            uint32_t f[4];
            ldsm_x4_at(f, k_at + np * row16 + kk * 32);
#pragma unroll
            for (int i = 0; i < HPW; ++i) {
              if (i > 0 && !one_group) ldsm_x4_at(f, k_of[i] + np * row16 + kk * 32);
              mma_bf16_16816(s[i][0], qa[i][kk], f[0], f[1]);
              mma_bf16_16816(s[i][1], qa[i][kk], f[2], f[3]);
            }
          }
        }
#pragma unroll
        for (int i = 0; i < HPW; ++i) {
          if (h0 + i >= H) continue;
#pragma unroll
          for (int ni = 0; ni < 2; ++ni) {
            *reinterpret_cast<float2*>(d + i * kMxHS + (np * 2 + ni) * 8) = make_float2(s[i][ni][0], s[i][ni][1]);
            *reinterpret_cast<float2*>(d + i * kMxHS + 8 * kMxLS + (np * 2 + ni) * 8) = make_float2(s[i][ni][2], s[i][ni][3]);
          }
        }
      }
    };
    auto scores = [&](int b) {
      const uint32_t kv = kv_at + (stages == 2 ? (b & 1) : 0) * stage_bytes;
      for (int hb = 0; hb < H; hb += hpb) {
        const int h0 = hb + warp * HPW;
        if (h0 >= H) break;
        if (H > hpb) {
#pragma unroll
          for (int i = 0; i < HPW; ++i) load_q(i, h0 + i);
        }
        if (HPW == 1 || (h0 + HPW - 1) / per == h0 / per) scores_of(kv, h0, std::true_type{});
        else scores_of(kv, h0, std::false_type{});
      }
    };
    auto weights = [&](int b, auto masked) {  // step 2; masked: some key of the block is hidden from some row of the tile
      const int k0 = b * kMxKeys;
      for (int nt = warp; nt < a.tile_rows * (kMxKeys / 8); nt += nw) {  // rows not in use: whatever their weights are, their sums are dropped
        const int r = nt / (kMxKeys / 8), ko = (nt % (kMxKeys / 8)) * 8;
        const float* src = S + r * kMxLS + ko + gq + 2 * tq * kMxHS;
        float z0[4] = {}, z1[4] = {}, z2[4] = {};  // the three terms in accumulators of their own: independent products in flight
#pragma unroll
        for (int kk = 0; kk < NK; ++kk) {
          if (NK == 1 || kk * 16 < H) {
            uint32_t hi[2], mid[2], lo[2];
            split3(src[kk * 16 * kMxHS], src[(kk * 16 + 1) * kMxHS], hi[0], mid[0], lo[0]);
            split3(src[(kk * 16 + 8) * kMxHS], src[(kk * 16 + 9) * kMxHS], hi[1], mid[1], lo[1]);
            mma_free(z0, ta[kk], hi[0], hi[1]);
            mma_free(z1, ta[kk], mid[0], mid[1]);
            mma_free(z2, ta[kk], lo[0], lo[1]);
          }
        }
        float w[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) w[e] = fast_logistic2(fmaf(z0[e] + (z1[e] + z2[e]), scale2, e < 2 ? bias_a : bias_b));
        if (masked) {
          const int seen = s_req[r] == rq ? s_pos[r] - k0 - ko - 2 * tq : -1;  // keys 2 tq + c of this group are visible for c <= seen
          if (seen < 0) w[0] = w[2] = 0.f;
          if (seen < 1) w[1] = w[3] = 0.f;
        }
        bf16* d = P + gq * kMxHP + r * kMxLP + ko + 2 * tq;  // (heads past the last one: weights that nobody reads)
        *reinterpret_cast<uint32_t*>(d) = pack_bf16(w[0], w[1]);
        *reinterpret_cast<uint32_t*>(d + 8 * kMxHP) = pack_bf16(w[2], w[3]);
      }
    };
    auto values_of = [&](uint32_t kv, int l0, auto one_group) {  // step 3 for the heads h_base + l0 and on
      const uint32_t v_at = kv + v_lane + (uint32_t)((h_base + l0) / per * vdim * 2);
      uint32_t v_of[HPW], p_of[HPW];
#pragma unroll
      for (int i = 0; i < HPW; ++i) {
        v_of[i] = kv + v_lane + (uint32_t)(min((h_base + l0 + i) / per, G - 1) * vdim * 2);
        p_of[i] = p_at + (uint32_t)(min(l0 + i, nh - 1) * kMxHP * 2);
      }
#pragma unroll
      for (int kk = 0; kk < kMxKeys / 16; ++kk) {
        uint32_t pa[HPW][4];
#pragma unroll
        for (int i = 0; i < HPW; ++i) ldsm_x4_at(pa[i], p_of[i] + kk * 32);
#pragma unroll
        for (int np = 0; np < DV / 16; ++np) {
          if (EXACT || np * 16 < vdim) {
            uint32_t f[4];
            ldsm_x4_trans_at(f, v_at + kk * row16 + np * 32);
#pragma unroll
            for (int i = 0; i < HPW; ++i) {
              if (i > 0 && !one_group) ldsm_x4_trans_at(f, v_of[i] + kk * row16 + np * 32);
              mma_bf16_16816(o[i][np * 2], pa[i], f[0], f[1]);
              mma_bf16_16816(o[i][np * 2 + 1], pa[i], f[2], f[3]);
            }
          }
        }
      }
    };
    auto values = [&](int b) {
      const uint32_t kv = kv_at + (stages == 2 ? (b & 1) : 0) * stage_bytes;
      const int l0 = warp * HPW;
      if (l0 >= nh) return;
      if (HPW == 1 || (h_base + l0 + HPW - 1) / per == (h_base + l0) / per) values_of(kv, l0, std::true_type{});
      else values_of(kv, l0, std::false_type{});
    };
    if (b0 < b_end) {
      __syncthreads();  // the previous request's readers are done with every buffer
      note(b0, page_of(b0));
      note(b0 + 1, page_of(b0 + 1));
      __syncthreads();
      load(b0);
      cp_async_wait_all();
      __syncthreads();
      scores(b0);
      for (int b = b0; b < b_end; ++b) {
        const bool more = b + 1 < b_end;
        __syncthreads();  // this block's scores are complete; nobody reads the other stage or the weights any more
        if (more && stages == 2) load(b + 1);
        const int page = page_of(b + 2);  // the lookup travels while the weights are made
        if (whole_tile && (b + 1) * kMxKeys <= p_min + 1) weights(b, std::false_type{});
        else weights(b, std::true_type{});
        note(b + 2, page);  // the offsets of block b were read before the barrier above
        if (stages == 2) cp_async_wait_all();
        __syncthreads();  // weights complete, block b + 1 has landed (two stages)
        values(b);
        if (more && stages == 1) {
          __syncthreads();
          load(b + 1);
          cp_async_wait_all();
          __syncthreads();
        }
        if (more) scores(b + 1);
      }
    }
    r_first = r_last + 1;
  }
  const int l0 = warp * HPW;
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    if (l0 + i >= nh) continue;
    const int h = h_base + l0 + i;
    float fa = a.out_scale, fb = a.out_scale;
    if (a.gate && a.splits == 1) {
      if (in_a) fa *= logistic_exact(a.gate[(size_t)row_a * a.gate_ld + h]);
      if (in_b) fb *= logistic_exact(a.gate[(size_t)row_b * a.gate_ld + h]);
    }
#pragma unroll
    for (int ni = 0; ni < DV / 8; ++ni) {
      const int c = ni * 8 + 2 * tq;
      if (c >= vdim) continue;
      if (a.splits > 1) {
        float* pa = a.part + (((size_t)split * a.T + row_a) * H + h) * vdim + c;
        float* pb = a.part + (((size_t)split * a.T + row_b) * H + h) * vdim + c;
        if (in_a) *reinterpret_cast<float2*>(pa) = make_float2(o[i][ni][0], o[i][ni][1]);
        if (in_b) *reinterpret_cast<float2*>(pb) = make_float2(o[i][ni][2], o[i][ni][3]);
      } else {
        bf16* out = static_cast<bf16*>(a.out);
        if (in_a) *reinterpret_cast<uint32_t*>(out + (size_t)row_a * a.out_ld + h * vdim + c) = pack_bf16(o[i][ni][0] * fa, o[i][ni][1] * fa);
        if (in_b) *reinterpret_cast<uint32_t*>(out + (size_t)row_b * a.out_ld + h * vdim + c) = pack_bf16(o[i][ni][2] * fb, o[i][ni][3] * fb);
      }
    }
  }
}

// out = out_scale * logistic(gate) * sum of the shares' partial sums.  CTA = 64 entries of one row x PG groups of shares; a group adds its shares
// in order and the groups are added in order, so the result does not depend on timing.
template <typename E, int PG>
__global__ void __launch_bounds__(64 * PG) mixed_attention_merge_kernel(MixedArgs a) {
  __shared__ float part[PG][64];
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int t = blockIdx.x, c = threadIdx.x & 63, grp = threadIdx.x >> 6, i = blockIdx.y * 64 + c, n = a.H * a.vdim;
  float s = 0.f;
  if (i < n) {
    const float* p = a.part + (size_t)t * n + i;
    const size_t step = (size_t)a.T * n;
    int sp = grp;
    for (; sp + 7 * PG < a.splits; sp += 8 * PG) {  // eight independent loads in flight
      float v[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) v[u] = p[(size_t)(sp + u * PG) * step];
#pragma unroll
      for (int u = 0; u < 8; ++u) s += v[u];
    }
    for (; sp < a.splits; sp += PG) s += p[(size_t)sp * step];
  }
  if (PG > 1) {
    part[grp][c] = s;
    __syncthreads();
    if (grp) return;
#pragma unroll
    for (int g = 1; g < PG; ++g) s += part[g][c];
  }
  if (i >= n) return;
  const float f = a.gate ? a.out_scale * logistic_exact(a.gate[(size_t)t * a.gate_ld + i / a.vdim]) : a.out_scale;
  static_cast<E*>(a.out)[(size_t)t * a.out_ld + i] = from_f<E>(s * f);
}

// the same for a few shares of many rows: four entries per thread, 16-byte loads
template <typename E>
__global__ void __launch_bounds__(256) mixed_attention_merge4_kernel(MixedArgs a) {
  pdl_wait();
  pdl_launch_dependents();  // the next kernel may start its launch; it waits for this grid to finish before it reads
  const int t = blockIdx.x, i = (blockIdx.y * 256 + threadIdx.x) * 4, n = a.H * a.vdim;
  if (i >= n) return;
  const float* p = a.part + (size_t)t * n + i;
  const size_t step = (size_t)a.T * n;
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int sp = 0; sp < a.splits; ++sp) {
    const float4 v = *reinterpret_cast<const float4*>(p + (size_t)sp * step);
    s.x += v.x, s.y += v.y, s.z += v.z, s.w += v.w;
  }
  const float f = a.gate ? a.out_scale * logistic_exact(a.gate[(size_t)t * a.gate_ld + i / a.vdim]) : a.out_scale;  // vdim is a multiple of 4
  E* o = static_cast<E*>(a.out) + (size_t)t * a.out_ld + i;
  if constexpr (sizeof(E) == 2) *reinterpret_cast<uint2*>(o) = make_uint2(pack_bf16(s.x * f, s.y * f), pack_bf16(s.z * f, s.w * f));
  else *reinterpret_cast<float4*>(o) = make_float4(s.x * f, s.y * f, s.z * f, s.w * f);
}

static inline void fit_splits(MixedArgs& a, float* ws, size_t ws_bytes) {  // partial sums must fit into the workspace
  const size_t one = (size_t)a.T * a.H * a.vdim * sizeof(float);
  if (!ws) a.splits = 1;
  while (a.splits > 1 && one * a.splits > ws_bytes) --a.splits;
  a.part = ws;
}

template <typename E>
static void launch_merge(const MixedArgs& a, cudaStream_t st) {
  const dim3 g(a.T, (a.H * a.vdim + 63) / 64);
  const bool four = a.vdim % 4 == 0 && a.out_ld % 4 == 0 && (reinterpret_cast<uintptr_t>(a.out) & (4 * sizeof(E) - 1)) == 0 &&
                    (reinterpret_cast<uintptr_t>(a.part) & 15) == 0;
  if (a.splits <= 8 && four) launch(mixed_attention_merge4_kernel<E>, dim3(a.T, (a.H * a.vdim + 1023) / 1024), dim3(256), 0, st, true, a);
  else if (a.splits > 8) launch(mixed_attention_merge_kernel<E, 8>, g, dim3(512), 0, st, true, a);
  else launch(mixed_attention_merge_kernel<E, 1>, g, dim3(64), 0, st, true, a);
}

template <int DQ, int DV, int HPW, int NK, bool EXACT>
static int launch_mixed_mma(MixedArgs a, int max_kv, float* ws, size_t ws_bytes, cudaStream_t st) {
  const int tok = a.G * (a.dim + a.vdim);
  const size_t stage = (size_t)kMxKeys * (tok + 8) * 2, rest = (size_t)((a.H + 15) / 16 * 16) * kMxHS * 4 + (size_t)16 * kMxHP * 2;
  const size_t limit = 220 * 1024;
  const int stages = 2 * stage + rest <= limit ? 2 : 1;
  if (stages * stage + rest > limit) return -2;
  static bool attr_set = false;  // per template instance
  if (!attr_set) {
    if (cudaFuncSetAttribute(mixed_attention_mma_kernel<DQ, DV, HPW, NK, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)limit) != cudaSuccess)
      return (int)cudaGetLastError();
    attr_set = true;
  }
  a.tile_rows = a.T < kMxRows ? 1 : kMxRows;  // decode steps: a CTA per row, or rows of several requests would be walked one after the other
  const int tiles = (a.T + a.tile_rows - 1) / a.tile_rows, slices = (a.H + 15) / 16;
  const int warps = std::min(8, (std::min(16, a.H) + HPW - 1) / HPW);
  constexpr int per_sm = DQ <= 64 && HPW == 1 ? 2 : 1;  // CTAs that share an SM (the kernel's launch bounds)
  // shares of the key axis: a long prompt's tiles in two (or four), so that the ones with the most keys do not run on alone; few tiles: a CTA for every SM; in
  // a prompt portion a share is at least four blocks
  const int span = max_kv > 0 ? max_kv : a.T, blocks = (span + kMxKeys - 1) / kMxKeys;
  const int want = a.tile_rows == 1 ? sm_count() / (tiles * slices) : std::max(2 * per_sm, 2 * per_sm * sm_count() / (tiles * slices));
  a.splits = std::max(1, std::min({want, a.tile_rows == 1 ? blocks : blocks / 4, 64}));
  fit_splits(a, ws, ws_bytes);
  launch(mixed_attention_mma_kernel<DQ, DV, HPW, NK, EXACT>, dim3(a.splits, tiles, slices), dim3(warps * 32), stages * stage + rest, st, true, a, stages);
  if (a.splits > 1) launch_merge<bf16>(a, st);
  return (int)cudaGetLastError();
}

template <typename E>
static int launch_mixed(MixedArgs a, int max_kv, float* ws, size_t ws_bytes, cudaStream_t st) {
  int kb = 32;
  while (kb > 4 && mixed_smem(a.H, a.G, a.dim, a.vdim, kb) > 100 * 1024) kb /= 2;
  const size_t smem = mixed_smem(a.H, a.G, a.dim, a.vdim, kb);
  if (smem > 200 * 1024) return -2;
  if (smem > 48 * 1024) {
    static bool attr_set = false;  // per template instance
    if (!attr_set) {
      if (cudaFuncSetAttribute(mixed_attention_kernel<E>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return (int)cudaGetLastError();
      attr_set = true;
    }
  }
  const int blocks = max_kv > 0 ? (max_kv + kb - 1) / kb : 1;
  a.splits = std::max(1, std::min({(2 * sm_count() + a.T - 1) / a.T, blocks, 128}));
  fit_splits(a, ws, ws_bytes);
  launch(mixed_attention_kernel<E>, dim3(a.T, a.splits), dim3(256), smem, st, true, a, kb);
  if (a.splits > 1) launch_merge<E>(a, st);
  return (int)cudaGetLastError();
}

}  // namespace pk

using namespace pk;

extern "C" int pk_gqa_mixed_attention(const void* q, const void* cache, const void* score_mix, const float* head_bias, const float* gate, int gate_ld,
                                      const int* positions, const int* req, const int* page_off, const int* pages, void* out, int out_ld,
                                      float out_scale, long page_stride, int page_size, int tokens, int heads, int kv_heads, int dim, int vdim,
                                      float scale, int max_kv_len, void* workspace, long workspace_bytes, int f32, pk_stream st) {
  if (!q || !cache || !positions || !req || !page_off || !pages || !out || tokens <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 ||
      vdim <= 0 || page_size <= 0 || out_ld < heads * vdim || max_kv_len < 0 || workspace_bytes < 0)
    return -1;
  MixedArgs a{q, cache, score_mix, head_bias, gate, positions, req, page_off, pages, out, nullptr, page_stride, gate_ld, out_ld, page_size, tokens, heads,
              kv_heads, dim, vdim, 1, kMxRows, scale, out_scale};
  const bool aligned = ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 3) == 0 &&
                       page_stride % 8 == 0 && out_ld % 2 == 0;
  if (!f32 && aligned && dim % 16 == 0 && vdim % 16 == 0 && dim <= 128 && vdim <= 128 && heads <= 16 * kMxMaxK) {
    int rc;
#define PK_MX(DQ, DV, EX)                                                                                                                  \
  (heads > 16  ? launch_mixed_mma<DQ, DV, 2, kMxMaxK, EX>(a, max_kv_len, static_cast<float*>(workspace), (size_t)workspace_bytes, st) \
   : heads > 8 ? launch_mixed_mma<DQ, DV, 2, 1, EX>(a, max_kv_len, static_cast<float*>(workspace), (size_t)workspace_bytes, st)       \
               : launch_mixed_mma<DQ, DV, 1, 1, EX>(a, max_kv_len, static_cast<float*>(workspace), (size_t)workspace_bytes, st))
    if (dim == 64 && vdim == 64) rc = PK_MX(64, 64, true);
    else if (dim == 128 && vdim == 128) rc = PK_MX(128, 128, true);
    else rc = PK_MX(128, 128, false);
#undef PK_MX
    if (rc != -2) return rc;
  }
  return f32 ? launch_mixed<float>(a, max_kv_len, static_cast<float*>(workspace), (size_t)workspace_bytes, st) : launch_mixed<bf16>(a, max_kv_len, static_cast<float*>(workspace), (size_t)workspace_bytes, st);
}
