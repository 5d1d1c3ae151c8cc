// Linear attention with a decaying matrix state for a RAGGED step.  Per head, with S [D, V] per sequence slot (fp32):
//     S_t = diag(w_t) S_(t-1) + k_t v_t^T        o_t = S_t^T q_t
// w_t is a number per head (fixed decay) or a vector per key channel made from the input,
//     w_t = sigmoid(z_t)^(1/tau),  z_t = A2 a_t + b     (a_t: a low-rank projection, columns of the projection row).
// q, k and v are columns of the packed projection row; options applied when they are read: SiLU on all three, rotation of
// the first rd dimensions of q and k (pairs (i, i + rd/2), host-made cos / sin table), factors on q and k.  Everything
// from there on is fp32.  An entry whose first position is 0 starts from a zero state whatever its slot held.
//
// Three forms of the same recurrence:
//   row by row      decode rows and short portions: a CTA owns 32 state columns of one (entry, head) in registers
//   blocks          portions of prompts: 16 rows at a time as small matrix products.  With c_t = log w_1 + .. + log w_t inside
//                   a block that starts from S_in:
//                     o_t   = S_in^T (e^(c_t) q_t) + sum_(s<=t) (sum_d q_t[d] k_s[d] e^(c_t[d] - c_s[d])) v_s
//                     S_out = diag(e^(c_L)) S_in + sum_s (e^(c_L - c_s) k_s) v_s^T
//                   Every exponent is <= 0.
//   tiles of 64 rows in parallel: what a tile adds to the state, an elementwise carry in order, read-outs; bf16 engines run
//                   the first and the last on the tensor cores (linear_attn_tc.cu)
#include <math.h>

#include "linear_attn.cuh"

namespace dli {

__device__ __forceinline__ float la_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// log w_t of key channel `ch` (head-major): (1/tau) log sigmoid(A2[ch] . a_t + b[ch])
template <typename E>
__device__ __forceinline__ float la_log_decay(const E* pr, int ch, const LinAttn& a) {
  const float* w = a.a2 + (size_t)ch * a.rank;
  float z = 0.f;
  for (int r = 0; r < a.rank; ++r) z = fmaf(w[r], l_to_f(pr[a.a_off + r]), z);
  return la_log_sigmoid(z + a.a2_b[ch]) * a.inv_tau;
}

// ---- row by row ---------------------------------------------------------------------------------------------------
constexpr int kLaCols = 32, kLaThreads = 256, kLaGroups = kLaThreads / (kLaCols / 4);

// Grid (entries, heads, ceil(V / 32)).  Thread (group, column quad): NR state rows group, group + 32, .. of 4 columns.
template <typename E, int NR>
__global__ void __launch_bounds__(kLaThreads)
linattn_rows_kernel(const E* __restrict__ proj, float* __restrict__ S, float* __restrict__ o, LinAttn a) {
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;                // [D]
  float* ks = qs + a.D;          // [D]
  float* ws = ks + a.D;          // [D]
  __shared__ float red[kLaThreads / 32][kLaCols];
  pdl_wait();
  pdl_trigger();
  const int4 e = reinterpret_cast<const int4*>(a.ent)[blockIdx.x];  // slot, first row, rows, first position
  const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int D = a.D, V = a.V;
  const int grp = tid >> 3, c0 = blockIdx.z * kLaCols + (tid & 7) * 4;
  const bool quad = (V & 3) == 0;
  float* Sp = S + ((size_t)e.x * a.H + h) * D * V;
  float s[NR][4];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = grp + i * kLaGroups;
    s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    if (e.w > 0 && d < D) {
      if (quad) {
        if (c0 < V) {
          const float4 f = *reinterpret_cast<const float4*>(Sp + (size_t)d * V + c0);
          s[i][0] = f.x; s[i][1] = f.y; s[i][2] = f.z; s[i][3] = f.w;
        }
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c0 + j < V) s[i][j] = Sp[(size_t)d * V + c0 + j];
      }
    }
  }
  const float wfix = a.log_decay ? expf(a.log_decay[h]) : 0.f;
  for (int t = 0; t < e.z; ++t) {
    const size_t row = (size_t)e.y + t;
    const E* pr = proj + row * a.ldp;
    for (int i = tid; i < D; i += kLaThreads) {
      qs[i] = la_qk(pr, a.q_off + h * D, i, a, e.w + t, a.q_scale);
      ks[i] = la_qk(pr, a.k_off + h * D, i, a, e.w + t, a.k_scale);
      ws[i] = a.log_decay ? wfix : expf(la_log_decay(pr, h * D + i, a));
    }
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float u = c0 + j < V ? l_to_f(pr[a.v_off + h * V + c0 + j]) : 0.f;
      v[j] = a.silu ? silu_f(u) : u;
    }
    __syncthreads();
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = grp + i * kLaGroups;
      if (d < D) {
        const float w = ws[d], k = ks[d], q = qs[d];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          s[i][j] = fmaf(w, s[i][j], k * v[j]);
          acc[j] = fmaf(s[i][j], q, acc[j]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], 8);
      acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], 16);
    }
    if (lane < 8) *reinterpret_cast<float4*>(&red[warp][lane * 4]) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    __syncthreads();
    if (tid < kLaCols) {
      float u = 0.f;
#pragma unroll
      for (int w = 0; w < kLaThreads / 32; ++w) u += red[w][tid];
      const int c = blockIdx.z * kLaCols + tid;
      if (c < V) o[row * ((size_t)a.H * V) + h * V + c] = u;
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = grp + i * kLaGroups;
    if (d < D) {
      if (quad) {
        if (c0 < V) *reinterpret_cast<float4*>(Sp + (size_t)d * V + c0) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c0 + j < V) Sp[(size_t)d * V + c0 + j] = s[i][j];
      }
    }
  }
}

// ---- log decays of every row (portions): lg [rows, H*D] -----------------------------------------------------------------
// 16 rows x 256 channels per CTA: a thread holds 16 entries of its channel's row of A2 at a time, the rows' a_t are in shared
// memory.
constexpr int kLdRows = 16;
template <typename E>
__global__ void __launch_bounds__(256)
linattn_log_decay_kernel(const E* __restrict__ proj, float* __restrict__ lg, LinAttn a, int rows) {
  __shared__ __align__(16) float as[kLdRows][16];
  pdl_wait();
  pdl_trigger();
  const int n = a.H * a.D, row0 = blockIdx.x * kLdRows, ch = blockIdx.y * 256 + threadIdx.x;
  float z[kLdRows];
  const float b = ch < n ? a.a2_b[ch] : 0.f;
#pragma unroll
  for (int t = 0; t < kLdRows; ++t) z[t] = 0.f;
  for (int r0 = 0; r0 < a.rank; r0 += 16) {
    __syncthreads();
    {
      const int t = threadIdx.x >> 4, r = r0 + (threadIdx.x & 15);
      as[t][threadIdx.x & 15] = (row0 + t < rows && r < a.rank) ? l_to_f(proj[(size_t)(row0 + t) * a.ldp + a.a_off + r]) : 0.f;
    }
    float w[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) w[r] = (ch < n && r0 + r < a.rank) ? a.a2[(size_t)ch * a.rank + r0 + r] : 0.f;
    __syncthreads();
#pragma unroll
    for (int t = 0; t < kLdRows; ++t)
#pragma unroll
      for (int r = 0; r < 16; r += 4) {
        const float4 f = *reinterpret_cast<const float4*>(&as[t][r]);
        z[t] = fmaf(w[r], f.x, z[t]); z[t] = fmaf(w[r + 1], f.y, z[t]); z[t] = fmaf(w[r + 2], f.z, z[t]); z[t] = fmaf(w[r + 3], f.w, z[t]);
      }
  }
  if (ch >= n) return;
#pragma unroll
  for (int t = 0; t < kLdRows; ++t)
    if (row0 + t < rows) lg[(size_t)(row0 + t) * n + ch] = la_log_sigmoid(z[t] + b) * a.inv_tau;
}

// ---- blocks -------------------------------------------------------------------------------------------------------------
constexpr int kLaL = 16;      // rows per block
constexpr int kLaP = 20;      // padded row of the transposed blocks
constexpr int kLaVc = 64;     // value columns per CTA

static inline size_t linattn_block_smem(int D, bool gated) {
  return sizeof(float) * ((size_t)D * kLaVc + 2 * (size_t)D * kLaP + (gated ? 3 : 2) * (size_t)kLaL * (D + 1) + kLaL * kLaVc +
                          kLaL * (kLaL + 1) + kLaL + 4);
}

//   mode 0: one CTA per (entry, head, 64 columns) walks the blocks in order;  mode 1: per tile, what it adds to the state;
//   mode 3: per tile, the outputs from the tile's incoming state (where mode 1 left its contribution and the carry put it)
template <typename E, int mode, bool gated>
__global__ void __launch_bounds__(256)
linattn_blocks_kernel(const E* __restrict__ proj, const float* __restrict__ lg, float* __restrict__ S, float* __restrict__ o,
                      LinAttn a, const int32_t* __restrict__ tiles, float* __restrict__ scr_u, float* __restrict__ scr_w) {
  extern __shared__ __align__(16) float sm[];
  const int D = a.D, V = a.V, DP = D + 1;
  float* qT = sm;                        // [D][kLaP]  e^(c_t) q_t
  float* kT = qT + D * kLaP;             // [D][kLaP]  e^(c_L - c_t) k_t
  float* St = kT + D * kLaP;             // [D][kLaVc]
  float* vs = St + D * kLaVc;            // [L][kLaVc]
  float* qs = vs + kLaL * kLaVc;         // [L][D+1]
  float* ks = qs + kLaL * DP;            // [L][D+1]
  float* cs = gated ? ks + kLaL * DP : ks;                 // [L][D+1]
  float* G = (gated ? cs : ks) + kLaL * DP;                // [L][L+1]
  float* pw = G + kLaL * (kLaL + 1);     // [L+1] powers of the fixed decay
  pdl_wait();
  pdl_trigger();
  const int ei = mode == 0 ? (int)blockIdx.x : tiles[2 * blockIdx.x];
  const int4 e = reinterpret_cast<const int4*>(a.ent)[ei];  // slot, first row, rows, first position
  const int h = blockIdx.y, v0 = blockIdx.z * kLaVc, tid = threadIdx.x;
  const int nv = min(kLaVc, V - v0);
  const size_t HD = (size_t)a.H * D;
  float* Sp = S + ((size_t)e.x * a.H + h) * D * V + v0;
  float* Up = mode == 0 ? nullptr : scr_u + ((size_t)blockIdx.x * a.H + h) * D * V + v0;
  const int vcol = tid & 63, tg = tid >> 6;
  for (int i = tid; i < D * kLaVc; i += 256) {
    const int d = i >> 6, v = i & 63;
    float s = 0.f;
    if (v < nv) {
      if (mode == 0 && e.w > 0) s = Sp[(size_t)d * V + v];
      if (mode == 3) s = Up[(size_t)d * V + v];
    }
    St[i] = s;
  }
  const float ld = gated ? 0.f : a.log_decay[h];
  if (!gated && tid <= kLaL) pw[tid] = tid == 0 ? 1.f : expf(ld * tid);
  const int b_first = mode == 0 ? 0 : tiles[2 * blockIdx.x + 1];
  const int b_end = mode == 0 ? e.z : min(e.z, b_first + kLaTile);
  float total[4] = {0.f, 0.f, 0.f, 0.f};  // mode 1, gated: the tile's summed log decay of channels tid, tid + 256, ..
  for (int b0 = b_first; b0 < b_end; b0 += kLaL) {
    const int nb = min(kLaL, b_end - b0);
    __syncthreads();
    for (int i = tid; i < kLaL * D; i += 256) {
      const int t = i / D, d = i - t * D;
      float q = 0.f, k = 0.f, c = 0.f;
      if (t < nb) {
        const size_t row = (size_t)(e.y + b0 + t);
        const E* pr = proj + row * a.ldp;
        const int pos = e.w + b0 + t;
        if (mode != 1) q = la_qk(pr, a.q_off + h * D, d, a, pos, a.q_scale);
        k = la_qk(pr, a.k_off + h * D, d, a, pos, a.k_scale);
        if (gated) c = lg[row * HD + h * D + d];
      }
      if (mode != 1) qs[t * DP + d] = q;
      ks[t * DP + d] = k;
      if (gated) cs[t * DP + d] = c;
    }
    for (int i = tid; i < kLaL * kLaVc; i += 256) {
      const int t = i >> 6, v = i & 63;
      float u = 0.f;
      if (t < nb && v < nv) {
        u = l_to_f(proj[(size_t)(e.y + b0 + t) * a.ldp + a.v_off + h * V + v0 + v]);
        if (a.silu) u = silu_f(u);
      }
      vs[i] = u;
    }
    __syncthreads();
    // running log decays of every channel, and the rows weighted for the read-out and for the state
    int n_own = 0;
    for (int d = tid; d < D; d += 256, ++n_own) {
      if (gated) {
        // c_L - c_t as the sum of the later rows' logarithms: a difference of running sums would lose the small ones
        // behind a fast decay
        float r = 0.f;
        for (int t = kLaL - 1; t >= 0; --t) {
          kT[d * kLaP + t] = ks[t * DP + d] * expf(r);
          r += cs[t * DP + d];
        }
        if (mode == 1 && n_own < 4) total[n_own] += r;
        float c = 0.f;
        for (int t = 0; t < kLaL; ++t) {
          c += cs[t * DP + d];
          cs[t * DP + d] = c;
          if (mode != 1) qT[d * kLaP + t] = qs[t * DP + d] * expf(c);
        }
      } else {
        for (int t = 0; t < kLaL; ++t) {
          if (mode != 1) qT[d * kLaP + t] = qs[t * DP + d] * pw[t + 1];
          kT[d * kLaP + t] = t < nb ? ks[t * DP + d] * pw[nb - 1 - t] : 0.f;
        }
      }
    }
    if (mode != 1) {
      const int t = tid >> 4, s = tid & 15;
      float g = 0.f;
      if (gated) __syncthreads();  // the running sums are complete
      if (s <= t) {
        if (gated) {
          for (int d = 0; d < D; ++d)
            g = fmaf(qs[t * DP + d] * ks[s * DP + d], expf(cs[t * DP + d] - cs[s * DP + d]), g);
        } else {
          for (int d = 0; d < D; ++d) g = fmaf(qs[t * DP + d], ks[s * DP + d], g);
          g *= pw[t - s];
        }
      }
      G[t * (kLaL + 1) + s] = g;
    }
    __syncthreads();
    if (mode != 1) {
      // rows 4 tg .. 4 tg + 3 of column vcol
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      for (int d = 0; d < D; ++d) {
        const float4 q4 = *reinterpret_cast<const float4*>(qT + d * kLaP + tg * 4);
        const float sv = St[d * kLaVc + vcol];
        acc[0] = fmaf(q4.x, sv, acc[0]); acc[1] = fmaf(q4.y, sv, acc[1]);
        acc[2] = fmaf(q4.z, sv, acc[2]); acc[3] = fmaf(q4.w, sv, acc[3]);
      }
#pragma unroll
      for (int s = 0; s < kLaL; ++s) {
        const float vv = vs[s * kLaVc + vcol];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i] = fmaf(G[(tg * 4 + i) * (kLaL + 1) + s], vv, acc[i]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = tg * 4 + i;
        if (t < nb && vcol < nv) o[(size_t)(e.y + b0 + t) * ((size_t)a.H * V) + h * V + v0 + vcol] = acc[i];
      }
      if (mode == 3 && b0 + kLaL >= b_end) break;  // no later block needs the state
      __syncthreads();                             // every read of the incoming state is done
    }
    {
      float vv[kLaL];
#pragma unroll
      for (int s = 0; s < kLaL; ++s) vv[s] = vs[s * kLaVc + vcol];
      const float wf = gated ? 0.f : pw[nb];
      for (int d = tg; d < D; d += 4) {
        const float w = gated ? expf(cs[(kLaL - 1) * DP + d]) : wf;
        float u = w * St[d * kLaVc + vcol];
#pragma unroll
        for (int s4 = 0; s4 < kLaL; s4 += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(kT + d * kLaP + s4);
          u = fmaf(k4.x, vv[s4], u); u = fmaf(k4.y, vv[s4 + 1], u); u = fmaf(k4.z, vv[s4 + 2], u); u = fmaf(k4.w, vv[s4 + 3], u);
        }
        St[d * kLaVc + vcol] = u;
      }
    }
  }
  if (mode == 3) return;
  __syncthreads();
  for (int i = tid; i < D * kLaVc; i += 256) {
    const int d = i >> 6, v = i & 63;
    if (v < nv) {
      if (mode == 0) Sp[(size_t)d * V + v] = St[i];
      else Up[(size_t)d * V + v] = St[i];
    }
  }
  if (mode == 1 && blockIdx.z == 0) {
    float* wp = scr_w + ((size_t)blockIdx.x * a.H + h) * D;
    int n_own = 0;
    for (int d = tid; d < D; d += 256, ++n_own) wp[d] = expf(gated ? total[min(n_own, 3)] : ld * (b_end - b_first));
  }
}

// The carry over an entry's tiles in order, elementwise: grid (entries, heads, ceil(D*V / 256)).
__global__ void __launch_bounds__(256)
linattn_carry_kernel(const int32_t* __restrict__ ent, const int32_t* __restrict__ tiles, int n_tiles, float* __restrict__ S,
                     float* __restrict__ scr_u, const float* __restrict__ scr_w, int H, int D, int V) {
  __shared__ int t_first;
  pdl_wait();
  pdl_trigger();
  const int4 e = reinterpret_cast<const int4*>(ent)[blockIdx.x];
  const int h = blockIdx.y;
  if (threadIdx.x == 0) {
    int t = 0;
    while (t < n_tiles && tiles[2 * t] != (int)blockIdx.x) ++t;
    t_first = t;
  }
  __syncthreads();
  const int NV = D * V, i = blockIdx.z * 256 + threadIdx.x;
  if (i >= NV) return;
  const int d = i / V, nt = (e.z + kLaTile - 1) / kLaTile;
  float* Sp = S + ((size_t)e.x * H + h) * NV + i;
  float s = e.w > 0 ? *Sp : 0.f;
  for (int c0 = 0; c0 < nt; c0 += 8) {  // eight tiles' contributions requested before the first is used
    float u[8], w[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const size_t t = (size_t)t_first + min(c0 + k, nt - 1);
      u[k] = scr_u[(t * H + h) * NV + i];
      w[k] = scr_w[(t * H + h) * D + d];
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      if (c0 + k >= nt) break;
      scr_u[(((size_t)t_first + c0 + k) * H + h) * NV + i] = s;
      s = fmaf(w[k], s, u[k]);
    }
  }
  *Sp = s;
}

template <typename E>
static int launch_rows(const void* proj, float* S, float* o, int n_ent, const LinAttn& a, cudaStream_t s) {
  const dim3 grid(n_ent, a.H, (a.V + kLaCols - 1) / kLaCols);
  const size_t smem = 3 * sizeof(float) * (size_t)a.D;
#define LA_ROWS(NR) DLI_LAUNCH("linattn_rows", (linattn_rows_kernel<E, NR>), grid, dim3(kLaThreads), smem, s, (const E*)proj, S, o, a)
  if (a.D <= kLaGroups) LA_ROWS(1);
  else if (a.D <= 2 * kLaGroups) LA_ROWS(2);
  else if (a.D <= 4 * kLaGroups) LA_ROWS(4);
  else if (a.D <= 8 * kLaGroups) LA_ROWS(8);
  else LA_ROWS(16);
#undef LA_ROWS
  return DLI_OK;
}

template <typename E, bool gated>
static int launch_blocks(const void* proj, float* lg, float* S, float* o, const LinAttn& a, int n_ent, int rows, const int32_t* tiles,
                         int n_tiles, float* scratch, cudaStream_t s) {
  const size_t smem = linattn_block_smem(a.D, gated);
  const int nz = (a.V + kLaVc - 1) / kLaVc;
  float* scr_u = scratch;
  float* scr_w = scratch ? scratch + (size_t)n_tiles * a.H * a.D * a.V : nullptr;
#define LA_BLOCKS(MODE, GX, WHAT)                                                                                              \
  do {                                                                                                                         \
    static PerDeviceOnce once;                                                                                                 \
    DLI_ONCE_PER_DEVICE(once, dev, DLI_CUDA_CALL(cudaFuncSetAttribute(linattn_blocks_kernel<E, MODE, gated>,                   \
                                                                       cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024))); \
    DLI_LAUNCH(WHAT, (linattn_blocks_kernel<E, MODE, gated>), dim3(GX, a.H, nz), dim3(256), smem, s, (const E*)proj, lg, S, o, a, \
               tiles, scr_u, scr_w);                                                                                           \
  } while (0)
  if (!scratch) {
    LA_BLOCKS(0, n_ent, "linattn_blocks");
    return DLI_OK;
  }
  const bool tc = sizeof(E) == 2 && lg && linattn_tc_supported(a);
  if (tc) {
    const int rc = linattn_tc_local(proj, lg, a, rows, tiles, n_tiles, scr_u, scr_w, s);
    if (rc != DLI_OK) return rc;
  } else {
    LA_BLOCKS(1, n_tiles, "linattn_local");
  }
  DLI_LAUNCH("linattn_carry", linattn_carry_kernel, dim3(n_ent, a.H, (a.D * a.V + 255) / 256), dim3(256), 0, s, a.ent, tiles, n_tiles,
             S, scr_u, (const float*)scr_w, a.H, a.D, a.V);
  if (tc) return linattn_tc_out(proj, lg, o, a, rows, tiles, n_tiles, scr_u, s);
  LA_BLOCKS(3, n_tiles, "linattn_out");
#undef LA_BLOCKS
  return DLI_OK;
}

}  // namespace dli

using namespace dli;

extern "C" {

int dli_linattn_tc_supported(int D, int V, int gated, int silu, int rd, int dt) {
  LinAttn a{};
  a.D = D; a.V = V; a.silu = silu; a.rd = rd;
  static const float one = 0.f;
  a.log_decay = gated ? nullptr : &one;
  return dt == 0 && linattn_tc_supported(a) ? 1 : 0;
}

size_t dli_linattn_scratch_floats(int n_tiles, int H, int D, int V) {
  return (size_t)n_tiles * H * D * ((size_t)V + 1);
}

int dli_linattn_ragged(const void* proj, float* S, float* o, const int32_t* ent, int n_ent, int rows, int H, int D, int V, int ldp,
                       int q_off, int k_off, int v_off, int silu, float q_scale, float k_scale, const float* cos_t,
                       const float* sin_t, int rd, const float* log_decay, int a_off, int rank, const float* a2, const float* a2_b,
                       float inv_tau, int blocked, float* lg, const int32_t* tiles, int n_tiles, float* scratch, int dt,
                       dli_stream_t stream) {
  DLI_CHECK_ARG(proj && S && o && ent && H > 0 && D > 0 && V > 0, "dli_linattn_ragged: null pointer or empty shape");
  DLI_CHECK_ARG(D <= 16 * kLaGroups, "dli_linattn_ragged: key size %d (at most %d)", D, 16 * kLaGroups);
  DLI_CHECK_ARG(rd >= 0 && rd <= D && rd % 2 == 0 && (rd == 0 || (cos_t && sin_t)), "dli_linattn_ragged: %d rotated dimensions of %d", rd, D);
  DLI_CHECK_ARG(log_decay || (a2 && a2_b && rank > 0 && a_off >= 0 && a_off + rank <= ldp),
                "dli_linattn_ragged: either a decay per head or the low-rank decay projection");
  DLI_CHECK_ARG(q_off >= 0 && k_off >= 0 && v_off >= 0 && q_off + H * D <= ldp && k_off + H * D <= ldp && v_off + H * V <= ldp,
                "dli_linattn_ragged: columns outside the projection row");
  DLI_CHECK_ARG((reinterpret_cast<uintptr_t>(ent) & 15u) == 0 && aligned16(S), "dli_linattn_ragged: ent and S must be 16-byte aligned");
  DLI_CHECK_ARG(dt == 0 || dt == 1, "element type %d: 0 = bf16, 1 = float", dt);
  if (n_ent <= 0 || rows <= 0) return DLI_OK;
  LinAttn a{ent, H, D, V, ldp, q_off, k_off, v_off, silu ? 1 : 0, q_scale, k_scale, cos_t, sin_t, rd, log_decay, a_off, rank, a2, a2_b,
            inv_tau};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool gated = log_decay == nullptr;
  if (!blocked || linattn_block_smem(D, gated) > 200 * 1024)
    return dt == 0 ? launch_rows<bf16>(proj, S, o, n_ent, a, s) : launch_rows<float>(proj, S, o, n_ent, a, s);
  if (gated) {
    DLI_CHECK_ARG(lg, "dli_linattn_ragged: portions with a decay per channel need scratch for the log decays");
    const dim3 grid((rows + kLdRows - 1) / kLdRows, (H * D + 255) / 256);
    if (dt == 0) DLI_LAUNCH("linattn_log_decay", linattn_log_decay_kernel<bf16>, grid, dim3(256), 0, s, (const bf16*)proj, lg, a, rows);
    else DLI_LAUNCH("linattn_log_decay", linattn_log_decay_kernel<float>, grid, dim3(256), 0, s, (const float*)proj, lg, a, rows);
  }
  float* scr = tiles && n_tiles > 0 ? scratch : nullptr;  // with scratch: all tiles in parallel
  if (dt == 0) return gated ? launch_blocks<bf16, true>(proj, lg, S, o, a, n_ent, rows, tiles, n_tiles, scr, s)
                            : launch_blocks<bf16, false>(proj, lg, S, o, a, n_ent, rows, tiles, n_tiles, scr, s);
  return gated ? launch_blocks<float, true>(proj, lg, S, o, a, n_ent, rows, tiles, n_tiles, scr, s)
               : launch_blocks<float, false>(proj, lg, S, o, a, n_ent, rows, tiles, n_tiles, scr, s);
}

}  // extern "C"
