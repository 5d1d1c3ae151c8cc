// Linear attention over portions of prompts on the tensor cores (bf16 engines): the per-tile passes of the tile-parallel
// form of linear_attn.cu, 64 rows of one (entry, head) and 64 value columns per CTA, m16n8k16 products with fp32
// accumulators.
//
//   local   U = sum_s (e^(c_L - c_s) k_s) v_s^T                    what the tile adds to the state
//   out     o_t = S_in^T (e^(c_t) q_t) + sum_(s<=t) g_ts v_s,  g_ts = sum_d q_t[d] k_s[d] e^(c_t[d] - c_s[d])
//
// The state, the decays and what enters the recurrence are fp32 quantities: an operand that is not exact in bf16 goes in as
// the sum of two bf16 numbers (16 bits of mantissa together) and a product of two such operands as three products, so the
// rounding of an operand is 2^-17 instead of 2^-9.
//
// Fixed decay: g_ts = w^(t-s) q_t . k_s, the weights are applied to the fp32 accumulators.  Decay per key channel: the
// weights belong on the operands.  For the 16-row block i with reference r = c before its first row, q_t e^(c_t - r) and
// k_s e^(r - c_s) of the earlier rows have exponents <= 0.  Inside the block r - c_s >= 0 is the block's own decay: below
// kSafeLog2 it is multiplied in all the same (bf16 has fp32's exponent range), above it the block's 16 x 16 scores are
// summed directly with e^(c_t - c_s) per channel.
#include <math.h>

#include "linear_attn.cuh"
#include "mma_utils.cuh"

namespace dli {

constexpr int kTcThreads = 128;
constexpr int kTcVc = 64;           // value columns per CTA
constexpr int kTcVp = kTcVc + 8;    // padded row (an odd number of 16-byte pieces: ldmatrix without bank conflicts)
constexpr float kSafeLog2 = 58.f;
constexpr float kLog2e = 1.4426950408889634f;

static inline size_t tc_local_smem(int D, bool gated) {
  return 2 * ((size_t)2 * kLaTile * (D + 8) + (size_t)(gated ? 1 : 2) * kLaTile * kTcVp);
}
static inline size_t tc_out_smem(int D, bool gated) {
  return 2 * ((size_t)(gated ? 2 : 4) * kLaTile * (D + 8) + (size_t)(gated ? 1 : 2) * kLaTile * kTcVp + (size_t)2 * D * kTcVp) +
         (gated ? 4 * (size_t)kLaTile * (D + 8) : 0);
}

bool linattn_tc_supported(const LinAttn& a) {
  const bool gated = a.log_decay == nullptr;
  return a.D % 16 == 0 && a.V % 8 == 0 && tc_out_smem(a.D, gated) <= 220 * 1024 && !(gated && (a.silu || a.rd));
}

__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - bf_lo(hi), y - bf_hi(hi));
}

// Rows of one tile: where they are, and how many.
struct TcTile {
  size_t row0;      // first row of the step
  int pos0, nb;     // its position, rows in the tile
};

// The prepared q or k (columns `base` ..) of the tile's rows as hi + lo (both [64][D+8]); rows past the tile: zeros.
// wexp: log2 of a factor per row step, applied as 2^(wexp * (nb - 1 - t)) (0: none).
__device__ __forceinline__ void stage_rows(const bf16* __restrict__ proj, int base, const LinAttn& a, const TcTile& tl, float scale,
                                           float wexp, bf16* __restrict__ hi, bf16* __restrict__ lo) {
  const int D = a.D, DP = D + 8, half = a.rd >> 1, np = D >> 1;
  for (int i = threadIdx.x; i < kLaTile * np; i += kTcThreads) {
    const int t = i / np, p = i - t * np;
    // a rotated pair (p, p + half), or two neighbours behind the rotated dimensions
    const bool hp = p < half;
    const int i0 = hp ? p : 2 * p, i1 = hp ? p + half : 2 * p + 1;
    float u = 0.f, v = 0.f;
    if (t < tl.nb) {
      const bf16* pr = proj + (tl.row0 + t) * a.ldp + base;
      u = __bfloat162float(pr[i0]);
      v = __bfloat162float(pr[i1]);
      if (a.silu) { u = silu_f(u); v = silu_f(v); }
      if (hp) {
        const size_t at = (size_t)(tl.pos0 + t) * half + p;
        const float c = a.cos_t[at], s = a.sin_t[at], u2 = u * c - v * s;
        v = v * c + u * s;
        u = u2;
      }
      const float f = wexp != 0.f ? scale * exp2f(wexp * (float)(tl.nb - 1 - t)) : scale;
      u *= f;
      v *= f;
    }
    uint32_t h, l;
    split2(u, v, h, l);
    bf16* hr = hi + t * DP;
    bf16* lr = lo + t * DP;
    if (hp) {
      hr[i0] = __ushort_as_bfloat16((unsigned short)(h & 0xffffu)); hr[i1] = __ushort_as_bfloat16((unsigned short)(h >> 16));
      lr[i0] = __ushort_as_bfloat16((unsigned short)(l & 0xffffu)); lr[i1] = __ushort_as_bfloat16((unsigned short)(l >> 16));
    } else {
      *reinterpret_cast<uint32_t*>(hr + i0) = h;
      *reinterpret_cast<uint32_t*>(lr + i0) = l;
    }
  }
}

// The rows' raw bf16 columns [64][n] (n a multiple of 8) into rows of `ld` elements, zeros past the tile and past n_valid.
__device__ __forceinline__ void stage_raw(const bf16* __restrict__ proj, int base, const LinAttn& a, const TcTile& tl, int n, int n_valid,
                                          bf16* __restrict__ dst, int ld) {
  const bool al = (a.ldp % 8 == 0) && (base % 8 == 0) && (reinterpret_cast<uintptr_t>(proj) & 15u) == 0;
  const int nc = n >> 3;
  for (int i = threadIdx.x; i < kLaTile * nc; i += kTcThreads) {
    const int t = i / nc, c = (i - t * nc) * 8;
    uint4 u = make_uint4(0, 0, 0, 0);
    if (t < tl.nb && c < n_valid) {
      const bf16* src = proj + (tl.row0 + t) * a.ldp + base + c;
      if (al) {
        u = ld_16B(src);
      } else {
        const unsigned short* us = reinterpret_cast<const unsigned short*>(src);
        u.x = us[0] | ((uint32_t)us[1] << 16); u.y = us[2] | ((uint32_t)us[3] << 16);
        u.z = us[4] | ((uint32_t)us[5] << 16); u.w = us[6] | ((uint32_t)us[7] << 16);
      }
    }
    *reinterpret_cast<uint4*>(dst + t * ld + c) = u;
  }
}

// v of the tile: gated: raw columns; fixed decay: SiLU if asked for, as hi + lo
template <bool gated>
__device__ __forceinline__ void stage_values(const bf16* __restrict__ proj, int h, int v0, const LinAttn& a, const TcTile& tl,
                                             bf16* __restrict__ vh, bf16* __restrict__ vl) {
  const int base = a.v_off + h * a.V + v0, nv = min(kTcVc, a.V - v0);
  if constexpr (gated) {
    stage_raw(proj, base, a, tl, kTcVc, nv, vh, kTcVp);
  } else {
    for (int i = threadIdx.x; i < kLaTile * (kTcVc / 2); i += kTcThreads) {
      const int t = i / (kTcVc / 2), c = 2 * (i % (kTcVc / 2));
      float x = 0.f, y = 0.f;
      if (t < tl.nb && c < nv) {
        const bf16* src = proj + (tl.row0 + t) * a.ldp + base + c;
        x = __bfloat162float(src[0]);
        y = __bfloat162float(src[1]);
        if (a.silu) { x = silu_f(x); y = silu_f(y); }
      }
      uint32_t hi, lo;
      split2(x, y, hi, lo);
      *reinterpret_cast<uint32_t*>(vh + t * kTcVp + c) = hi;
      *reinterpret_cast<uint32_t*>(vl + t * kTcVp + c) = lo;
    }
  }
}

// ---- what a tile adds to the state: U [D, 64 columns] -------------------------------------------------------------------
template <bool gated>
__global__ void __launch_bounds__(kTcThreads)
linattn_tc_local_kernel(const bf16* __restrict__ proj, const float* __restrict__ lg, LinAttn a, const int32_t* __restrict__ tiles,
                        float* __restrict__ scr_u, float* __restrict__ scr_w) {
  extern __shared__ __align__(16) uint8_t sm_raw[];
  const int D = a.D, DP = D + 8;
  bf16* kh = reinterpret_cast<bf16*>(sm_raw);   // [64][D+8] k_s e^(c_L - c_s), hi
  bf16* kl = kh + kLaTile * DP;                 // lo
  bf16* vh = kl + kLaTile * DP;                 // [64][72]
  bf16* vl = vh + kLaTile * kTcVp;              // fixed decay only
  pdl_wait();
  pdl_trigger();
  const int4 e = reinterpret_cast<const int4*>(a.ent)[tiles[2 * blockIdx.x]];  // slot, first row, rows, first position
  const int b0 = tiles[2 * blockIdx.x + 1], h = blockIdx.y, v0 = blockIdx.z * kTcVc;
  const TcTile tl{(size_t)(e.y + b0), e.w + b0, min(kLaTile, e.z - b0)};
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* wp = scr_w + ((size_t)blockIdx.x * a.H + h) * D;
  stage_values<gated>(proj, h, v0, a, tl, vh, vl);
  if constexpr (gated) {
    // a thread per channel walks the rows from the last to the first: c_L - c_s is the sum of the later rows' log decays
    for (int d = tid; d < D; d += kTcThreads) {
      float r = 0.f;
      const float* lp = lg + tl.row0 * ((size_t)a.H * D) + h * D + d;
      const bf16* kp = proj + tl.row0 * a.ldp + a.k_off + h * D + d;
      for (int t0 = kLaTile - 8; t0 >= 0; t0 -= 8) {
        float l8[8], k8[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const int t = t0 + u;
          l8[u] = t < tl.nb ? lp[(size_t)t * a.H * D] * kLog2e : 0.f;
          k8[u] = t < tl.nb ? __bfloat162float(kp[(size_t)t * a.ldp]) * a.k_scale : 0.f;
        }
#pragma unroll
        for (int u = 7; u >= 0; --u) {
          const float x = k8[u] * ex2_ftz(r);
          r += l8[u];
          const bf16 hi = __float2bfloat16_rn(x);
          kh[(t0 + u) * DP + d] = hi;
          kl[(t0 + u) * DP + d] = __float2bfloat16_rn(x - __bfloat162float(hi));
        }
      }
      if (blockIdx.z == 0) wp[d] = ex2_ftz(r);
    }
  } else {
    const float l2 = a.log_decay[h] * kLog2e;
    stage_rows(proj, a.k_off + h * D, a, tl, a.k_scale, l2, kh, kl);
    if (blockIdx.z == 0)
      for (int d = tid; d < D; d += kTcThreads) wp[d] = exp2f(l2 * (float)tl.nb);
  }
  __syncthreads();
  const uint32_t skh = smem_u32(kh), skl = smem_u32(kl), svh = smem_u32(vh), svl = smem_u32(vl);
  const int mi = lane >> 3, r8 = lane & 7, gq = lane >> 2, t4 = lane & 3;
  const int nv = min(kTcVc, a.V - v0);
  float* Up = scr_u + (((size_t)blockIdx.x * a.H + h) * D) * a.V + v0;
  for (int mt = warp; mt < D / 16; mt += 4) {
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t ah[4], al[4];
      const uint32_t aoff = ((ks * 16 + (mi >> 1) * 8 + r8) * DP + mt * 16 + (mi & 1) * 8) * 2;
      ldmatrix_x4_trans(ah, skh + aoff);
      ldmatrix_x4_trans(al, skl + aoff);
#pragma unroll
      for (int jp = 0; jp < 4; ++jp) {
        uint32_t vf[4];
        const uint32_t voff = ((ks * 16 + (mi & 1) * 8 + r8) * kTcVp + jp * 16 + (mi >> 1) * 8) * 2;
        ldmatrix_x4_trans(vf, svh + voff);
        mma_16816(acc[2 * jp], ah, vf[0], vf[1]);
        mma_16816(acc[2 * jp + 1], ah, vf[2], vf[3]);
        mma_16816(acc[2 * jp], al, vf[0], vf[1]);
        mma_16816(acc[2 * jp + 1], al, vf[2], vf[3]);
        if constexpr (!gated) {
          ldmatrix_x4_trans(vf, svl + voff);
          mma_16816(acc[2 * jp], ah, vf[0], vf[1]);
          mma_16816(acc[2 * jp + 1], ah, vf[2], vf[3]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = j * 8 + 2 * t4;
      if (c < nv) {
#pragma unroll
        for (int r = 0; r < 2; ++r)
          *reinterpret_cast<float2*>(Up + (size_t)(mt * 16 + gq + 8 * r) * a.V + c) = make_float2(acc[j][2 * r], acc[j][2 * r + 1]);
      }
    }
  }
}

// ---- read-outs ----------------------------------------------------------------------------------------------------------
// Warp w owns rows 16 w .. 16 w + 15 of the tile and all 64 columns; its keys are the 16-row blocks 0 .. w.
template <bool gated>
__global__ void __launch_bounds__(kTcThreads)
linattn_tc_out_kernel(const bf16* __restrict__ proj, const float* __restrict__ lg, float* __restrict__ o, LinAttn a,
                      const int32_t* __restrict__ tiles, const float* __restrict__ scr_u) {
  extern __shared__ __align__(16) uint8_t sm_raw[];
  const int D = a.D, DP = D + 8;
  bf16* qh = reinterpret_cast<bf16*>(sm_raw);        // [64][D+8]
  bf16* kh = qh + kLaTile * DP;
  bf16* ql = kh + kLaTile * DP;                      // fixed decay only: the lo parts
  bf16* kl = gated ? ql : ql + kLaTile * DP;
  bf16* vh = gated ? ql : kl + kLaTile * DP;         // [64][72]
  bf16* vl = vh + kLaTile * kTcVp;                   // fixed decay only
  bf16* sh = gated ? vl : vl + kLaTile * kTcVp;      // [D][72] the incoming state, hi and lo
  bf16* sl = sh + D * kTcVp;
  float* C = reinterpret_cast<float*>(sl + D * kTcVp);  // [64][D+8] gated: running log2 decays, inclusive
  pdl_wait();
  pdl_trigger();
  const int4 e = reinterpret_cast<const int4*>(a.ent)[tiles[2 * blockIdx.x]];  // slot, first row, rows, first position
  const int b0 = tiles[2 * blockIdx.x + 1], h = blockIdx.y, v0 = blockIdx.z * kTcVc;
  const TcTile tl{(size_t)(e.y + b0), e.w + b0, min(kLaTile, e.z - b0)};
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int nv = min(kTcVc, a.V - v0);
  stage_values<gated>(proj, h, v0, a, tl, vh, vl);
  if constexpr (gated) {
    stage_raw(proj, a.q_off + h * D, a, tl, D, D, qh, DP);
    stage_raw(proj, a.k_off + h * D, a, tl, D, D, kh, DP);
    for (int d = tid; d < D; d += kTcThreads) {
      float c = 0.f;
      const float* lp = lg + tl.row0 * ((size_t)a.H * D) + h * D + d;
      for (int t0 = 0; t0 < kLaTile; t0 += 8) {
        float l8[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) l8[u] = t0 + u < tl.nb ? lp[(size_t)(t0 + u) * a.H * D] * kLog2e : 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) { c += l8[u]; C[(t0 + u) * DP + d] = c; }
      }
    }
  } else {
    stage_rows(proj, a.q_off + h * D, a, tl, a.q_scale, 0.f, qh, ql);
    stage_rows(proj, a.k_off + h * D, a, tl, a.k_scale, 0.f, kh, kl);
  }
  const float* Sp = scr_u + (((size_t)blockIdx.x * a.H + h) * D) * a.V + v0;
  for (int i = tid; i < D * (kTcVc / 4); i += kTcThreads) {
    const int d = i / (kTcVc / 4), c = 4 * (i % (kTcVc / 4));
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < nv) f = *reinterpret_cast<const float4*>(Sp + (size_t)d * a.V + c);
    uint2 hi, lo;
    split2(f.x, f.y, hi.x, lo.x);
    split2(f.z, f.w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(sh + d * kTcVp + c) = hi;
    *reinterpret_cast<uint2*>(sl + d * kTcVp + c) = lo;
  }
  __syncthreads();
  if (warp * 16 >= tl.nb) return;  // no rows for this warp (no barrier follows)

  const uint32_t sqh = smem_u32(qh), sql = smem_u32(ql), skh = smem_u32(kh), skl = smem_u32(kl), svh = smem_u32(vh), svl = smem_u32(vl),
                 ssh = smem_u32(sh), ssl = smem_u32(sl);
  const int mi = lane >> 3, r8 = lane & 7, gq = lane >> 2, t4 = lane & 3;
  const int trow[2] = {warp * 16 + gq, warp * 16 + gq + 8};
  const float* Cr = gated ? C + (warp * 16 - 1) * DP : nullptr;  // the reference row (before the warp's first; warp 0: zeros)

  // does the block's own decay leave the range in which it can be multiplied in?
  bool direct = false;
  if constexpr (gated) {
    float worst = 0.f;
    for (int d = lane; d < D; d += 32) worst = fmaxf(worst, (warp > 0 ? Cr[d] : 0.f) - C[(warp * 16 + 15) * DP + d]);
    direct = warp_max(worst) > kSafeLog2;
  }

  float acc[8][4];   // S_in^T q, then everything
  float g[4][2][4];  // scores: key block j, key octet, fragment
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int n = 0; n < 2; ++n) g[j][n][0] = g[j][n][1] = g[j][n][2] = g[j][n][3] = 0.f;

  for (int kk = 0; kk < D / 16; ++kk) {
    uint32_t ah[4], al[4];     // the rows' operand of the state product
    uint32_t gh[4], gl[4];     // ... and of the scores
    float2 cr[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
    const uint32_t aoff = ((warp * 16 + (mi & 1) * 8 + r8) * DP + kk * 16 + (mi >> 1) * 8) * 2;
    ldmatrix_x4(ah, sqh + aoff);
    if constexpr (gated) {
      // fragment x: row trow[x & 1], channels kk*16 + (x >> 1)*8 + 2 t4 and the next
      if (warp > 0) {
        cr[0] = *reinterpret_cast<const float2*>(Cr + kk * 16 + 2 * t4);
        cr[1] = *reinterpret_cast<const float2*>(Cr + kk * 16 + 8 + 2 * t4);
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float2 c = *reinterpret_cast<const float2*>(C + trow[x & 1] * DP + kk * 16 + (x >> 1) * 8 + 2 * t4);
        const float2 r = cr[x >> 1];
        const float u = bf_lo(ah[x]), v = bf_hi(ah[x]);
        split2(u * ex2_ftz(c.x - r.x), v * ex2_ftz(c.y - r.y), gh[x], gl[x]);
        split2(u * ex2_ftz(c.x), v * ex2_ftz(c.y), ah[x], al[x]);
      }
    } else {
      ldmatrix_x4(al, sql + aoff);
#pragma unroll
      for (int x = 0; x < 4; ++x) { gh[x] = ah[x]; gl[x] = al[x]; }
    }
#pragma unroll
    for (int jp = 0; jp < 4; ++jp) {
      uint32_t bh[4], bl[4];
      const uint32_t soff = ((kk * 16 + (mi & 1) * 8 + r8) * kTcVp + jp * 16 + (mi >> 1) * 8) * 2;
      ldmatrix_x4_trans(bh, ssh + soff);
      ldmatrix_x4_trans(bl, ssl + soff);
      mma_16816(acc[2 * jp], ah, bh[0], bh[1]);
      mma_16816(acc[2 * jp + 1], ah, bh[2], bh[3]);
      mma_16816(acc[2 * jp], ah, bl[0], bl[1]);
      mma_16816(acc[2 * jp + 1], ah, bl[2], bl[3]);
      mma_16816(acc[2 * jp], al, bh[0], bh[1]);
      mma_16816(acc[2 * jp + 1], al, bh[2], bh[3]);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j > warp || (j == warp && direct)) continue;
      uint32_t bh[4], bl[4];
      const uint32_t koff = ((j * 16 + (mi >> 1) * 8 + r8) * DP + kk * 16 + (mi & 1) * 8) * 2;
      ldmatrix_x4(bh, skh + koff);
      if constexpr (gated) {
        // fragment x: key row j*16 + (x >> 1)*8 + gq, channels kk*16 + (x & 1)*8 + 2 t4 and the next
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float2 c = *reinterpret_cast<const float2*>(C + (j * 16 + (x >> 1) * 8 + gq) * DP + kk * 16 + (x & 1) * 8 + 2 * t4);
          const float2 r = cr[x & 1];
          split2(bf_lo(bh[x]) * ex2_ftz(r.x - c.x), bf_hi(bh[x]) * ex2_ftz(r.y - c.y), bh[x], bl[x]);
        }
      } else {
        ldmatrix_x4(bl, skl + koff);
      }
      mma_16816(g[j][0], gh, bh[0], bh[1]);
      mma_16816(g[j][1], gh, bh[2], bh[3]);
      mma_16816(g[j][0], gh, bl[0], bl[1]);
      mma_16816(g[j][1], gh, bl[2], bl[3]);
      mma_16816(g[j][0], gl, bh[0], bh[1]);
      mma_16816(g[j][1], gl, bh[2], bh[3]);
    }
  }
  const float l2 = gated ? 0.f : a.log_decay[h] * kLog2e;
  if constexpr (gated) {
    if (direct) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j != warp) continue;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int t = trow[x >> 1], s = j * 16 + n * 8 + 2 * t4 + (x & 1);
            float u = 0.f;
            if (s <= t)
              for (int d = 0; d < D; ++d)
                u = fmaf(__bfloat162float(qh[t * DP + d]) * __bfloat162float(kh[s * DP + d]), ex2_ftz(C[t * DP + d] - C[s * DP + d]), u);
            g[j][n][x] = u;
          }
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[i][x] *= a.q_scale;
  } else {
    const float f0 = exp2f(l2 * (float)(trow[0] + 1)), f1 = exp2f(l2 * (float)(trow[1] + 1));
#pragma unroll
    for (int i = 0; i < 8; ++i) { acc[i][0] *= f0; acc[i][1] *= f0; acc[i][2] *= f1; acc[i][3] *= f1; }
  }
  // weights and the causal mask on the scores, then their product with the values
  const float gs = gated ? a.q_scale * a.k_scale : 1.f;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    if (j > warp) continue;
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      float w[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int back = trow[x >> 1] - (j * 16 + n * 8 + 2 * t4 + (x & 1));
        w[x] = back < 0 ? 0.f : g[j][n][x] * (gated ? gs : exp2f(l2 * (float)back));
      }
      split2(w[0], w[1], ph[2 * n], pl[2 * n]);
      split2(w[2], w[3], ph[2 * n + 1], pl[2 * n + 1]);
    }
#pragma unroll
    for (int jp = 0; jp < 4; ++jp) {
      uint32_t vf[4];
      const uint32_t voff = ((j * 16 + (mi & 1) * 8 + r8) * kTcVp + jp * 16 + (mi >> 1) * 8) * 2;
      ldmatrix_x4_trans(vf, svh + voff);
      mma_16816(acc[2 * jp], ph, vf[0], vf[1]);
      mma_16816(acc[2 * jp + 1], ph, vf[2], vf[3]);
      mma_16816(acc[2 * jp], pl, vf[0], vf[1]);
      mma_16816(acc[2 * jp + 1], pl, vf[2], vf[3]);
      if constexpr (!gated) {
        ldmatrix_x4_trans(vf, svl + voff);
        mma_16816(acc[2 * jp], ph, vf[0], vf[1]);
        mma_16816(acc[2 * jp + 1], ph, vf[2], vf[3]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    if (trow[r] >= tl.nb) continue;
    float* orow = o + (tl.row0 + trow[r]) * ((size_t)a.H * a.V) + h * a.V + v0;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = j * 8 + 2 * t4;
      if (c < nv) *reinterpret_cast<float2*>(orow + c) = make_float2(acc[j][2 * r], acc[j][2 * r + 1]);
    }
  }
}

template <bool gated>
static int tc_local(const void* proj, const float* lg, const LinAttn& a, const int32_t* tiles, int n_tiles, float* scr_u, float* scr_w,
                    cudaStream_t s) {
  static PerDeviceOnce once;
  DLI_ONCE_PER_DEVICE(once, dev, DLI_CUDA_CALL(cudaFuncSetAttribute(linattn_tc_local_kernel<gated>,
                                                                     cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)));
  DLI_LAUNCH("linattn_tc_local", linattn_tc_local_kernel<gated>, dim3(n_tiles, a.H, (a.V + kTcVc - 1) / kTcVc), dim3(kTcThreads),
             tc_local_smem(a.D, gated), s, (const bf16*)proj, lg, a, tiles, scr_u, scr_w);
  return DLI_OK;
}

template <bool gated>
static int tc_out(const void* proj, const float* lg, float* o, const LinAttn& a, const int32_t* tiles, int n_tiles, const float* scr_u,
                  cudaStream_t s) {
  static PerDeviceOnce once;
  DLI_ONCE_PER_DEVICE(once, dev, DLI_CUDA_CALL(cudaFuncSetAttribute(linattn_tc_out_kernel<gated>,
                                                                     cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)));
  DLI_LAUNCH("linattn_tc_out", linattn_tc_out_kernel<gated>, dim3(n_tiles, a.H, (a.V + kTcVc - 1) / kTcVc), dim3(kTcThreads),
             tc_out_smem(a.D, gated), s, (const bf16*)proj, lg, o, a, tiles, scr_u);
  return DLI_OK;
}

int linattn_tc_local(const void* proj, const float* lg, const LinAttn& a, const int32_t* tiles, int n_tiles, float* scr_u,
                     float* scr_w, cudaStream_t s) {
  return a.log_decay ? tc_local<false>(proj, lg, a, tiles, n_tiles, scr_u, scr_w, s)
                     : tc_local<true>(proj, lg, a, tiles, n_tiles, scr_u, scr_w, s);
}

int linattn_tc_out(const void* proj, const float* lg, float* o, const LinAttn& a, const int32_t* tiles, int n_tiles,
                   const float* scr_u, cudaStream_t s) {
  return a.log_decay ? tc_out<false>(proj, lg, o, a, tiles, n_tiles, scr_u, s) : tc_out<true>(proj, lg, o, a, tiles, n_tiles, scr_u, s);
}

}  // namespace dli
