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
//
// The key dimension goes through shared memory 64 channels at a time, so that several CTAs share an SM and one's loads
// overlap another's products.  With a fixed decay, q, k and v are prepared once per row by linattn_prep_kernel (SiLU,
// rotation, factors) and split into hi and lo rows there.
#include <math.h>

#include "linear_attn.cuh"
#include "mma_utils.cuh"

namespace dli {

constexpr int kTcThreads = 128;
constexpr int kTcVc = 64;           // value columns per CTA
constexpr int kTcVp = kTcVc + 8;    // padded row (an odd number of 16-byte pieces: ldmatrix without bank conflicts)
constexpr float kSafeLog2 = 58.f;
constexpr float kLog2e = 1.4426950408889634f;

constexpr int kTcDc = 64;           // key channels per pass
constexpr int kTcDp = kTcDc + 8;
constexpr int kTcRows = kLaTile * kTcDp;  // elements of one [64][72] block

static inline size_t tc_local_smem(bool gated) { return 2 * (size_t)kTcRows * (gated ? 3 : 4); }
static inline size_t tc_out_smem(bool gated) { return gated ? 2 * (size_t)kTcRows * 5 + 4 * (size_t)kTcRows : 2 * (size_t)kTcRows * 8; }

bool linattn_tc_supported(const LinAttn& a) {
  return a.D % 16 == 0 && a.V % 8 == 0 && !(a.log_decay == nullptr && (a.silu || a.rd));
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

// ---- fixed decay: q | k | v of every row, prepared, as a row of hi and a row of lo parts [2HD + HV] each ----------------
// An item is W consecutive dimensions of a head, with the W partners half a rotation away where they are rotated.
struct LinPrep {
  const int32_t* ent;
  const int32_t* tiles;
  bf16* hi;
  bf16* lo;
};

template <int W>
__global__ void __launch_bounds__(256)
linattn_prep_kernel(const bf16* __restrict__ proj, LinAttn a, LinPrep p) {
  pdl_wait();
  pdl_trigger();
  // one CTA per (tile, 8 of its rows)
  const int4 e = reinterpret_cast<const int4*>(p.ent)[p.tiles[2 * blockIdx.x]];  // slot, first row, rows, first position
  const int b0 = p.tiles[2 * blockIdx.x + 1] + 8 * blockIdx.y;
  const int nb = min(8, e.z - b0);
  const int half = a.rd >> 1, nrot = half / W, nqk = nrot + (a.D - a.rd) / W, nv = a.V / W;
  const int per_row = a.H * (2 * nqk + nv), C = a.H * (2 * a.D + a.V);
  for (int i = threadIdx.x; i < nb * per_row; i += 256) {
    const int t = i / per_row;
    int it = i - t * per_row;
    const size_t row = (size_t)(e.y + b0 + t);
    // which of q, k, v; head; item within the head
    const int part = it < a.H * nqk ? 0 : (it < 2 * a.H * nqk ? 1 : 2);
    it -= part == 0 ? 0 : (part == 1 ? a.H * nqk : 2 * a.H * nqk);
    const int n = part == 2 ? nv : nqk, sz = part == 2 ? a.V : a.D;
    const int h = it / n, x = it - h * n;
    const bool rot = part < 2 && x < nrot;
    const int d0 = part == 2 ? x * W : (rot ? x * W : a.rd + (x - nrot) * W);
    const int off = part == 0 ? a.q_off : (part == 1 ? a.k_off : a.v_off);
    const bf16* src = proj + row * a.ldp + off + h * sz + d0;
    const size_t dst = row * C + (part == 0 ? 0 : (part == 1 ? a.H * a.D : 2 * a.H * a.D)) + h * sz + d0;
    const float f = part == 0 ? a.q_scale : (part == 1 ? a.k_scale : 1.f);
    float u[W], v[W];
    auto load = [&](const bf16* s, float (&r)[W]) {
      if constexpr (W == 8) unpack8(ld_16B(s), r);
      else r[0] = __bfloat162float(*s);
      if (a.silu) {
#pragma unroll
        for (int k = 0; k < W; ++k) r[k] = silu_f(r[k]);
      }
    };
    auto store = [&](size_t at, const float (&r)[W]) {
      float l[W];
#pragma unroll
      for (int k = 0; k < W; ++k) l[k] = r[k] - round_bf16(r[k]);
      if constexpr (W == 8) {
        st_16B(p.hi + at, pack8(r));
        st_16B(p.lo + at, pack8(l));
      } else {
        p.hi[at] = __float2bfloat16_rn(r[0]);
        p.lo[at] = __float2bfloat16_rn(l[0]);
      }
    };
    load(src, u);
    if (rot) {
      load(src + half, v);
      const size_t tb = (size_t)(e.w + b0 + t) * half + d0;
#pragma unroll
      for (int k = 0; k < W; ++k) {
        const float c = a.cos_t[tb + k], s = a.sin_t[tb + k];
        const float u2 = (u[k] * c - v[k] * s) * f;
        v[k] = (v[k] * c + u[k] * s) * f;
        u[k] = u2;
      }
      store(dst, u);
      store(dst + half, v);
    } else {
#pragma unroll
      for (int k = 0; k < W; ++k) u[k] *= f;
      store(dst, u);
    }
  }
}

// 64 columns of the tile's rows (row stride ld, the first n_valid exist) into a [64][72] block; zeros elsewhere.  The copies
// are asynchronous where the rows' alignment allows: cp_async_wait before the barrier.
__device__ __forceinline__ void stage_raw(const bf16* __restrict__ src, size_t ld, const TcTile& tl, int n_valid, bool al, bf16* __restrict__ dst) {
  const uint32_t sd = smem_u32(dst);
#pragma unroll
  for (int i = threadIdx.x; i < kLaTile * 8; i += kTcThreads) {
    const int t = i >> 3, c = (i & 7) * 8;
    const bool ok = t < tl.nb && c < n_valid;
    const bf16* s = src + (ok ? t * ld + c : 0);
    if (al) {
      cp_async_16B(sd + (t * kTcDp + c) * 2, s, ok ? 16 : 0);
    } else {
      uint4 u = make_uint4(0, 0, 0, 0);
      if (ok) {
        const unsigned short* us = reinterpret_cast<const unsigned short*>(s);
        u.x = us[0] | ((uint32_t)us[1] << 16); u.y = us[2] | ((uint32_t)us[3] << 16);
        u.z = us[4] | ((uint32_t)us[5] << 16); u.w = us[6] | ((uint32_t)us[7] << 16);
      }
      *reinterpret_cast<uint4*>(dst + t * kTcDp + c) = u;
    }
  }
}

// may 8 consecutive columns from `base` on be copied as 16 bytes?
__device__ __forceinline__ bool raw_aligned(const bf16* p, size_t ld, int base) {
  return ld % 8 == 0 && base % 8 == 0 && (reinterpret_cast<uintptr_t>(p) & 15u) == 0;
}

// ---- what a tile adds to the state: U [D, 64 columns] -------------------------------------------------------------------
// Fixed decay: the weights w^(L-1-s) go onto the values (all channels share them); decay per channel: onto the keys.
template <bool gated>
__global__ void __launch_bounds__(kTcThreads)
linattn_tc_local_kernel(const bf16* __restrict__ proj, const bf16* __restrict__ hi, const bf16* __restrict__ lo,
                        const float* __restrict__ lg, LinAttn a, const int32_t* __restrict__ tiles, float* __restrict__ scr_u,
                        float* __restrict__ scr_w) {
  extern __shared__ __align__(16) uint8_t sm_raw[];
  const int D = a.D;
  bf16* kh = reinterpret_cast<bf16*>(sm_raw);   // [64][72] keys, hi
  bf16* kl = kh + kTcRows;                      // lo
  bf16* vh = kl + kTcRows;                      // [64][72] values
  bf16* vl = vh + kTcRows;                      // fixed decay only
  pdl_wait();
  pdl_trigger();
  const int4 e = reinterpret_cast<const int4*>(a.ent)[tiles[2 * blockIdx.x]];  // slot, first row, rows, first position
  const int b0 = tiles[2 * blockIdx.x + 1], h = blockIdx.y, v0 = blockIdx.z * kTcVc;
  const TcTile tl{(size_t)(e.y + b0), e.w + b0, min(kLaTile, e.z - b0)};
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int nv = min(kTcVc, a.V - v0), C = a.H * (2 * D + a.V);
  float* wp = scr_w + ((size_t)blockIdx.x * a.H + h) * D;
  const float l2 = gated ? 0.f : a.log_decay[h] * kLog2e;
  if constexpr (gated) {
    const int base = a.v_off + h * a.V + v0;
    stage_raw(proj + tl.row0 * a.ldp + base, a.ldp, tl, nv, raw_aligned(proj, a.ldp, base), vh);
  } else {
    const size_t at = tl.row0 * C + 2 * a.H * D + h * a.V + v0;
    for (int i = tid; i < kLaTile * 8; i += kTcThreads) {
      const int t = i >> 3, c = (i & 7) * 8;
      float x[8], y[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) x[k] = y[k] = 0.f;
      if (t < tl.nb && c < nv) {
        unpack8(ld_16B(hi + at + (size_t)t * C + c), x);
        unpack8(ld_16B(lo + at + (size_t)t * C + c), y);
        const float f = ex2_ftz(l2 * (float)(tl.nb - 1 - t));
#pragma unroll
        for (int k = 0; k < 8; ++k) { x[k] = (x[k] + y[k]) * f; y[k] = x[k] - round_bf16(x[k]); }
      }
      st_16B(vh + t * kTcDp + c, pack8(x));
      st_16B(vl + t * kTcDp + c, pack8(y));
    }
    if (blockIdx.z == 0)
      for (int d = tid; d < D; d += kTcThreads) wp[d] = exp2f(l2 * (float)tl.nb);
  }
  const uint32_t skh = smem_u32(kh), skl = smem_u32(kl), svh = smem_u32(vh), svl = smem_u32(vl);
  const int mi = lane >> 3, r8 = lane & 7, gq = lane >> 2, t4 = lane & 3;
  float* Up = scr_u + (((size_t)blockIdx.x * a.H + h) * D) * a.V + v0;
  for (int d0 = 0; d0 < D; d0 += kTcDc) {
    const int nd = min(kTcDc, D - d0);
    if (d0) __syncthreads();  // the previous pass's keys have been used
    if constexpr (gated) {
      // two threads per channel (rows 0..31 and 32..63) walk their rows from the last to the first: c_L - c_s is the sum of
      // the later rows' log decays; the earlier half adds the later half's total
      const int d = tid & 63, part = tid >> 6;
      const bool ok = d < nd;
      const float* lp = lg + tl.row0 * ((size_t)a.H * D) + h * D + d0 + d;
      const bf16* kp = proj + tl.row0 * a.ldp + a.k_off + h * D + d0 + d;
      float r = 0.f;
      if (part == 0 && ok)
        for (int t = 32; t < tl.nb; ++t) r += lp[(size_t)t * a.H * D] * kLog2e;
      for (int t0 = part * 32 + 24; t0 >= part * 32; t0 -= 8) {
        float l8[8], k8[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const int t = t0 + u;
          const bool in = ok && t < tl.nb;
          l8[u] = in ? lp[(size_t)t * a.H * D] * kLog2e : 0.f;
          k8[u] = in ? __bfloat162float(kp[(size_t)t * a.ldp]) * a.k_scale : 0.f;
        }
#pragma unroll
        for (int u = 7; u >= 0; --u) {
          const float x = k8[u] * ex2_ftz(r);
          r += l8[u];
          const bf16 xh = __float2bfloat16_rn(x);
          kh[(t0 + u) * kTcDp + d] = xh;
          kl[(t0 + u) * kTcDp + d] = __float2bfloat16_rn(x - __bfloat162float(xh));
        }
      }
      if (blockIdx.z == 0 && part == 0 && ok) wp[d0 + d] = ex2_ftz(r);
    } else {
      const size_t at = tl.row0 * C + a.H * D + h * D + d0;
      stage_raw(hi + at, C, tl, nd, true, kh);
      stage_raw(lo + at, C, tl, nd, true, kl);
    }
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
    if (warp * 16 >= nd) continue;
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t ah[4], al[4];
      const uint32_t aoff = ((ks * 16 + (mi >> 1) * 8 + r8) * kTcDp + warp * 16 + (mi & 1) * 8) * 2;
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
          *reinterpret_cast<float2*>(Up + (size_t)(d0 + warp * 16 + gq + 8 * r) * a.V + c) = make_float2(acc[j][2 * r], acc[j][2 * r + 1]);
      }
    }
  }
}

// ---- read-outs ----------------------------------------------------------------------------------------------------------
// Warp w owns rows 16 w .. 16 w + 15 of the tile and all 64 columns; its keys are the 16-row blocks 0 .. w.
template <bool gated>
__global__ void __launch_bounds__(kTcThreads, 3)
linattn_tc_out_kernel(const bf16* __restrict__ proj, const bf16* __restrict__ hi, const bf16* __restrict__ lo,
                      const float* __restrict__ lg, float* __restrict__ o, LinAttn a, const int32_t* __restrict__ tiles,
                      const float* __restrict__ scr_u) {
  extern __shared__ __align__(16) uint8_t sm_raw[];
  const int D = a.D;
  bf16* qh = reinterpret_cast<bf16*>(sm_raw);        // [64][72] blocks of 64 channels (values: 64 columns)
  bf16* kh = qh + kTcRows;
  bf16* vh = kh + kTcRows;
  bf16* sh = vh + kTcRows;                           // the incoming state, hi and lo
  bf16* sl = sh + kTcRows;
  bf16* ql = sl + kTcRows;                           // fixed decay only: the lo parts
  bf16* kl = ql + kTcRows;
  bf16* vl = kl + kTcRows;
  float* Cs = reinterpret_cast<float*>(sl + kTcRows);  // gated: [64][72] running log2 decays, inclusive
  pdl_wait();
  pdl_trigger();
  const int4 e = reinterpret_cast<const int4*>(a.ent)[tiles[2 * blockIdx.x]];  // slot, first row, rows, first position
  const int b0 = tiles[2 * blockIdx.x + 1], h = blockIdx.y, v0 = blockIdx.z * kTcVc;
  const TcTile tl{(size_t)(e.y + b0), e.w + b0, min(kLaTile, e.z - b0)};
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int nv = min(kTcVc, a.V - v0), C = a.H * (2 * D + a.V);
  if constexpr (gated) {
    const int base = a.v_off + h * a.V + v0;
    stage_raw(proj + tl.row0 * a.ldp + base, a.ldp, tl, nv, raw_aligned(proj, a.ldp, base), vh);
  } else {
    const size_t at = tl.row0 * C + 2 * a.H * D + h * a.V + v0;
    stage_raw(hi + at, C, tl, nv, true, vh);
    stage_raw(lo + at, C, tl, nv, true, vl);
  }
  const uint32_t sqh = smem_u32(qh), sql = smem_u32(ql), skh = smem_u32(kh), skl = smem_u32(kl), svh = smem_u32(vh), svl = smem_u32(vl),
                 ssh = smem_u32(sh), ssl = smem_u32(sl);
  const int mi = lane >> 3, r8 = lane & 7, gq = lane >> 2, t4 = lane & 3;
  const int trow[2] = {warp * 16 + gq, warp * 16 + gq + 8};
  float acc[8][4];   // S_in^T q, then everything
  float g[4][2][4];  // scores: key block j, key octet, fragment
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int n = 0; n < 2; ++n) g[j][n][0] = g[j][n][1] = g[j][n][2] = g[j][n][3] = 0.f;

  const float* Sp = scr_u + (((size_t)blockIdx.x * a.H + h) * D) * a.V + v0;
  const bool alq = raw_aligned(proj, a.ldp, a.q_off + h * D), alk = raw_aligned(proj, a.ldp, a.k_off + h * D);
  for (int d0 = 0; d0 < D; d0 += kTcDc) {
    const int nd = min(kTcDc, D - d0);
    if (d0) __syncthreads();  // the previous pass's blocks have been used
    if constexpr (gated) {
      stage_raw(proj + tl.row0 * a.ldp + a.q_off + h * D + d0, a.ldp, tl, nd, alq, qh);
      stage_raw(proj + tl.row0 * a.ldp + a.k_off + h * D + d0, a.ldp, tl, nd, alk, kh);
    } else {
      const size_t at = tl.row0 * C + h * D + d0;
      stage_raw(hi + at, C, tl, nd, true, qh);
      stage_raw(lo + at, C, tl, nd, true, ql);
      stage_raw(hi + at + a.H * D, C, tl, nd, true, kh);
      stage_raw(lo + at + a.H * D, C, tl, nd, true, kl);
    }
    cp_async_commit();
    if constexpr (gated) {
      // two threads per channel: rows 0..31, and rows 32..63 after the first half's total
      const int d = tid & 63, part = tid >> 6;
      const bool ok = d < nd;
      const float* lp = lg + tl.row0 * ((size_t)a.H * D) + h * D + d0 + d;
      float c = 0.f;
      if (part == 1 && ok)
        for (int t = 0; t < min(32, tl.nb); ++t) c += lp[(size_t)t * a.H * D] * kLog2e;
      for (int t0 = part * 32; t0 < part * 32 + 32; t0 += 8) {
        float l8[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) l8[u] = ok && t0 + u < tl.nb ? lp[(size_t)(t0 + u) * a.H * D] * kLog2e : 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) { c += l8[u]; Cs[(t0 + u) * kTcDp + d] = c; }
      }
    }
    for (int i = tid; i < kTcDc * (kTcVc / 4); i += kTcThreads) {
      const int d = i / (kTcVc / 4), c = 4 * (i % (kTcVc / 4));
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < nv && d < nd) f = *reinterpret_cast<const float4*>(Sp + (size_t)(d0 + d) * a.V + c);
      uint2 fh, fl;
      split2(f.x, f.y, fh.x, fl.x);
      split2(f.z, f.w, fh.y, fl.y);
      *reinterpret_cast<uint2*>(sh + d * kTcVp + c) = fh;
      *reinterpret_cast<uint2*>(sl + d * kTcVp + c) = fl;
    }
    cp_async_wait<0>();
    __syncthreads();
    if (warp * 16 >= tl.nb) continue;  // no rows for this warp
    // gated: the reference row of the warp's scores (the one before its first; warp 0: zeros), and whether its own block's
    // decay in this pass's channels leaves the range in which it can be multiplied in
    const float* Cr = Cs + (warp > 0 ? warp * 16 - 1 : 0) * kTcDp;
    bool direct = false;
    if constexpr (gated) {
      float worst = 0.f;
      for (int d = lane; d < nd; d += 32) worst = fmaxf(worst, (warp > 0 ? Cr[d] : 0.f) - Cs[(warp * 16 + 15) * kTcDp + d]);
      direct = warp_max(worst) > kSafeLog2;
    }
    for (int kk = 0; kk < nd / 16; ++kk) {
      uint32_t ah[4], al[4];     // the rows' operand of the state product
      uint32_t gh[4], gl[4];     // ... and of the scores
      float2 cr[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
      const uint32_t aoff = ((warp * 16 + (mi & 1) * 8 + r8) * kTcDp + kk * 16 + (mi >> 1) * 8) * 2;
      ldmatrix_x4(ah, sqh + aoff);
      if constexpr (gated) {
        // fragment x: row trow[x & 1], channels kk*16 + (x >> 1)*8 + 2 t4 and the next
        if (warp > 0) {
          cr[0] = *reinterpret_cast<const float2*>(Cr + kk * 16 + 2 * t4);
          cr[1] = *reinterpret_cast<const float2*>(Cr + kk * 16 + 8 + 2 * t4);
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float2 c = *reinterpret_cast<const float2*>(Cs + trow[x & 1] * kTcDp + kk * 16 + (x >> 1) * 8 + 2 * t4);
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
        const uint32_t koff = ((j * 16 + (mi >> 1) * 8 + r8) * kTcDp + kk * 16 + (mi & 1) * 8) * 2;
        ldmatrix_x4(bh, skh + koff);
        if constexpr (gated) {
          // fragment x: key row j*16 + (x >> 1)*8 + gq, channels kk*16 + (x & 1)*8 + 2 t4 and the next
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const float2 c = *reinterpret_cast<const float2*>(Cs + (j * 16 + (x >> 1) * 8 + gq) * kTcDp + kk * 16 + (x & 1) * 8 + 2 * t4);
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
                for (int d = 0; d < nd; ++d)
                  u = fmaf(__bfloat162float(qh[t * kTcDp + d]) * __bfloat162float(kh[s * kTcDp + d]),
                           ex2_ftz(Cs[t * kTcDp + d] - Cs[s * kTcDp + d]), u);
              g[j][n][x] += u;
            }
        }
      }
    }
  }  // passes over the key channels
  if (warp * 16 >= tl.nb) return;
  const float l2 = gated ? 0.f : a.log_decay[h] * kLog2e;
  if constexpr (gated) {
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

// fixed decay: the prepared rows in `prep` (hi rows, then lo rows; 2HD + HV floats' worth of bf16 pairs per row)
static LinPrep prep_rows(float* prep, const LinAttn& a, int rows, const int32_t* tiles) {
  bf16* hi = reinterpret_cast<bf16*>(prep);
  return LinPrep{a.ent, tiles, hi, hi + (size_t)rows * a.H * (2 * a.D + a.V)};
}

static int tc_prep(const void* proj, const LinAttn& a, const LinPrep& p, int n_tiles, cudaStream_t s) {
  const int half = a.rd / 2;
  const bool wide = half % 8 == 0 && (a.D - a.rd) % 8 == 0 && a.D % 8 == 0 && a.V % 8 == 0 && a.ldp % 8 == 0 && a.q_off % 8 == 0 &&
                    a.k_off % 8 == 0 && a.v_off % 8 == 0 && aligned16(proj) && aligned16(p.hi);
  const dim3 grid(n_tiles, kLaTile / 8);
  if (wide) DLI_LAUNCH("linattn_prep", linattn_prep_kernel<8>, grid, dim3(256), 0, s, (const bf16*)proj, a, p);
  else DLI_LAUNCH("linattn_prep", linattn_prep_kernel<1>, grid, dim3(256), 0, s, (const bf16*)proj, a, p);
  return DLI_OK;
}

#define TC_LAUNCH(KERNEL, SMEM, ...)                                                                                      \
  do {                                                                                                                    \
    static PerDeviceOnce once;                                                                                            \
    DLI_ONCE_PER_DEVICE(once, dev, DLI_CUDA_CALL(cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                                       (int)(SMEM))));                                    \
    DLI_LAUNCH(#KERNEL, KERNEL, dim3(n_tiles, a.H, (a.V + kTcVc - 1) / kTcVc), dim3(kTcThreads), SMEM, s, __VA_ARGS__);     \
  } while (0)

int linattn_tc_local(const void* proj, float* row_scr, const LinAttn& a, int rows, const int32_t* tiles, int n_tiles, float* scr_u,
                     float* scr_w, cudaStream_t s) {
  if (a.log_decay) {
    const LinPrep p = prep_rows(row_scr, a, rows, tiles);
    const int rc = tc_prep(proj, a, p, n_tiles, s);
    if (rc != DLI_OK) return rc;
    TC_LAUNCH(linattn_tc_local_kernel<false>, tc_local_smem(false), (const bf16*)proj, p.hi, p.lo, nullptr, a, tiles, scr_u, scr_w);
  } else {
    TC_LAUNCH(linattn_tc_local_kernel<true>, tc_local_smem(true), (const bf16*)proj, nullptr, nullptr, row_scr, a, tiles, scr_u, scr_w);
  }
  return DLI_OK;
}

int linattn_tc_out(const void* proj, float* row_scr, float* o, const LinAttn& a, int rows, const int32_t* tiles, int n_tiles,
                   const float* scr_u, cudaStream_t s) {
  if (a.log_decay) {
    const LinPrep p = prep_rows(row_scr, a, rows, tiles);
    TC_LAUNCH(linattn_tc_out_kernel<false>, tc_out_smem(false), (const bf16*)proj, p.hi, p.lo, nullptr, o, a, tiles, scr_u);
  } else {
    TC_LAUNCH(linattn_tc_out_kernel<true>, tc_out_smem(true), (const bf16*)proj, nullptr, nullptr, row_scr, o, a, tiles, scr_u);
  }
  return DLI_OK;
}

}  // namespace dli
