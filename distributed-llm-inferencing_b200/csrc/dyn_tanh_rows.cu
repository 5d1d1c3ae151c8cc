// Row-wise pieces of layers whose norms are DYNAMIC TANH maps, D(z) = tanh(alpha z) * w + b per channel, on a ragged step
// (fp32 residual stream).  Such a map needs no mean or variance of the row, so everything between two projections is
// elementwise:
//
//   x <- x + mult * D_post(y) (+ add)          y the sublayer's result, add e.g. the embedding output before a loop's next pass
//   h  = D_next(x)                             the next sublayer's input, fp32 and / or element type
//
// dli_dyn_tanh_close does both in one pass.  Without a router the grid is cut into column blocks of a few rows, a thread
// keeping its channels' weights in registers over the rows.  Where the norm feeds a mixture of experts, the router runs in
// the same kernel on the rows just made: a CTA takes one row (few rows) or four, whose normed values stay in shared memory,
// so that a router weight is read once for four rows.
#include "common.cuh"
#include "moe_route.cuh"

namespace dli {

struct DynTanh {
  const float* w;         // [d]
  const float* b;         // [d]
  float alpha;
};

struct DynTanhClose {
  DynTanh post;           // on the sublayer's result
  float mult;
  const float* add;       // [rows, d] or NULL
  DynTanh next;           // w NULL: no norm follows
  float* out_f;           // [rows, d] or NULL
  int rows, d;
};

template <int VEC> struct Chan { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Chan<VEC> ch_ld(const float* p) {
  Chan<VEC> r;
  if constexpr (VEC == 4) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    r.v[0] = u.x; r.v[1] = u.y; r.v[2] = u.z; r.v[3] = u.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int VEC> __device__ __forceinline__ Chan<VEC> ch_ld(const bf16* p) {
  Chan<VEC> r;
  if constexpr (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    r.v[0] = bf_lo(u.x); r.v[1] = bf_hi(u.x); r.v[2] = bf_lo(u.y); r.v[3] = bf_hi(u.y);
  } else {
    r.v[0] = __bfloat162float(*p);
  }
  return r;
}
template <int VEC> __device__ __forceinline__ void ch_st(float* p, const Chan<VEC>& r) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int VEC> __device__ __forceinline__ void ch_st(bf16* p, const Chan<VEC>& r) {
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(r.v[0], r.v[1]), pack_bf16(r.v[2], r.v[3]));
  else *p = __float2bfloat16_rn(r.v[0]);
}

// the weights of VEC channels of both maps
template <int VEC> struct ChanWeights { Chan<VEC> pw, pb, nw, nb; };
template <int VEC>
__device__ __forceinline__ ChanWeights<VEC> ch_weights(const DynTanhClose& a, int c, bool has_y) {
  ChanWeights<VEC> k;
  if (has_y) { k.pw = ch_ld<VEC>(a.post.w + c); k.pb = ch_ld<VEC>(a.post.b + c); }
  if (a.next.w) { k.nw = ch_ld<VEC>(a.next.w + c); k.nb = ch_ld<VEC>(a.next.b + c); }
  return k;
}
// the residual update of VEC channels
template <int VEC>
__device__ __forceinline__ void ch_update(Chan<VEC>& x, const Chan<VEC>& y, const ChanWeights<VEC>& k, const DynTanhClose& a) {
#pragma unroll
  for (int i = 0; i < VEC; ++i) x.v[i] = fmaf(a.mult, fmaf(tanhf(a.post.alpha * y.v[i]), k.pw.v[i], k.pb.v[i]), x.v[i]);
}
template <int VEC>
__device__ __forceinline__ Chan<VEC> ch_norm(const Chan<VEC>& x, const ChanWeights<VEC>& k, const DynTanhClose& a) {
  Chan<VEC> h;
#pragma unroll
  for (int i = 0; i < VEC; ++i) h.v[i] = fmaf(tanhf(a.next.alpha * x.v[i]), k.nw.v[i], k.nb.v[i]);
  return h;
}

// Grid (column blocks, groups of R rows); all loads of the group's rows are in flight before the first is used.
template <typename E, int VEC, int R>
__global__ void __launch_bounds__(256)
dyn_tanh_close_kernel(const E* __restrict__ y, float* __restrict__ x, E* __restrict__ out_e, DynTanhClose a) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  const bool on = c < a.d;
  ChanWeights<VEC> k;
  if (on) k = ch_weights<VEC>(a, c, y != nullptr);  // weights: not written by any kernel, read before the wait
  pdl_wait();
  pdl_trigger();
  if (!on) return;
  const int r0 = blockIdx.y * R;
  Chan<VEC> xv[R], yv[R], av[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    if (r0 + r >= a.rows) break;
    const size_t o = (size_t)(r0 + r) * a.d + c;
    xv[r] = ch_ld<VEC>(x + o);
    if (y) yv[r] = ch_ld<VEC>(y + o);
    if (a.add) av[r] = ch_ld<VEC>(a.add + o);
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    if (r0 + r >= a.rows) break;
    const size_t o = (size_t)(r0 + r) * a.d + c;
    if (y) ch_update<VEC>(xv[r], yv[r], k, a);
    if (a.add) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) xv[r].v[i] += av[r].v[i];
    }
    if (y || a.add) ch_st<VEC>(x + o, xv[r]);
    if (a.next.w) {
      const Chan<VEC> h = ch_norm<VEC>(xv[r], k, a);
      if (a.out_f) ch_st<VEC>(a.out_f + o, h);
      if (out_e) ch_st<VEC>(out_e + o, h);
    }
  }
}

// With the router: a CTA makes R rows, keeps the normed ones in shared memory [R][d] and forms the R x n_out logits with a
// warp per two outputs; then a warp per row chooses.  Behind the rows: R times the router's scratch.
template <typename E, int VEC, int R>
__global__ void __launch_bounds__(1024)
dyn_tanh_close_route_kernel(const E* __restrict__ y, float* __restrict__ x, E* __restrict__ out_e, DynTanhClose a, RouteArgs ra) {
  extern __shared__ __align__(16) float hs[];
  pdl_wait();
  pdl_trigger();
  const int d = a.d, ld = (d + 3) / 4 * 4, r0 = blockIdx.x * R, nr = min(R, a.rows - r0);
  for (int c = threadIdx.x * VEC; c < d; c += blockDim.x * VEC) {
    const ChanWeights<VEC> k = ch_weights<VEC>(a, c, y != nullptr);
    Chan<VEC> xv[R], yv[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      if (r >= nr) break;
      const size_t o = (size_t)(r0 + r) * d + c;
      xv[r] = ch_ld<VEC>(x + o);
      if (y) yv[r] = ch_ld<VEC>(y + o);
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      if (r >= nr) break;
      const size_t o = (size_t)(r0 + r) * d + c;
      if (y) ch_update<VEC>(xv[r], yv[r], k, a);
      if (a.add) {
        const Chan<VEC> av = ch_ld<VEC>(a.add + o);
#pragma unroll
        for (int i = 0; i < VEC; ++i) xv[r].v[i] += av.v[i];
      }
      if (y || a.add) ch_st<VEC>(x + o, xv[r]);
      const Chan<VEC> h = ch_norm<VEC>(xv[r], k, a);
      if (a.out_f) ch_st<VEC>(a.out_f + o, h);
      if (out_e) ch_st<VEC>(out_e + o, h);
      ch_st<VEC>(hs + r * ld + c, h);
    }
  }
  float* zs = hs + R * ld;
  const int zl = moe_route_floats(ra.n_out, ra.groups);
  if constexpr (R == 1) {
    __syncthreads();
    moe_route_row(hs, d, r0, ra, zs);
  } else {
    for (int r = nr; r < R; ++r)
      for (int c = threadIdx.x; c < d; c += blockDim.x) hs[r * ld + c] = 0.f;  // missing rows of the last group
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int n_log = ra.n_out + (ra.sg_w ? 1 : 0);
    auto weights_of = [&](int o) { return o < ra.n_out ? ra.wr + (size_t)o * d : ra.sg_w; };
    for (int o = 2 * warp; o < n_log; o += 2 * nw) {
      const int o1 = min(o + 1, n_log - 1);
      const float* __restrict__ w0 = weights_of(o);
      const float* __restrict__ w1 = weights_of(o1);
      float s0[R], s1[R];
#pragma unroll
      for (int r = 0; r < R; ++r) s0[r] = s1[r] = 0.f;
#pragma unroll 2
      for (int c = lane * VEC; c < d; c += 32 * VEC) {
        const Chan<VEC> u0 = ch_ld<VEC>(w0 + c), u1 = ch_ld<VEC>(w1 + c);
#pragma unroll
        for (int r = 0; r < R; ++r) {
          const Chan<VEC> h = ch_ld<VEC>(hs + r * ld + c);
#pragma unroll
          for (int i = 0; i < VEC; ++i) { s0[r] = fmaf(h.v[i], u0.v[i], s0[r]); s1[r] = fmaf(h.v[i], u1.v[i], s1[r]); }
        }
      }
#pragma unroll
      for (int r = 0; r < R; ++r) {
        s0[r] = warp_sum(s0[r]);
        s1[r] = warp_sum(s1[r]);
      }
      if (lane < 2 && o + lane < n_log) {
        const int q = o + lane;
#pragma unroll
        for (int r = 0; r < R; ++r) {
          const float z = lane ? s1[r] : s0[r];
          if (q < ra.n_out) zs[r * zl + q] = z + (ra.zb ? ra.zb[q] : 0.f);
          else zs[r * zl + 2 * ra.n_out + ra.groups] = z;
        }
      }
    }
    __syncthreads();
    if (warp < nr) moe_route_choose((size_t)r0 + warp, ra, zs + warp * zl);
  }
}

constexpr int kDytRouteRows = 4;             // rows per CTA of the routing form (steps of more than kDytFewRows rows)
constexpr int kDytFewRows = 64;
constexpr size_t kDytRouteMaxSmem = 96 * 1024;

template <typename E, int VEC>
static int launch_dyt(const void* y, float* x, void* out_e, const DynTanhClose& a, const RouteArgs* ra, cudaStream_t s) {
  if (!ra) {
    const int cols = (a.d + VEC - 1) / VEC;
    const int th = cols >= 256 ? 256 : (cols + 31) / 32 * 32;
    const int gx = (cols + th - 1) / th;
    if (a.rows > kDytFewRows) {
      DLI_LAUNCH("dyn_tanh_close", (dyn_tanh_close_kernel<E, VEC, 4>), dim3(gx, (a.rows + 3) / 4), dim3(th), 0, s, (const E*)y, x, (E*)out_e, a);
    } else {
      DLI_LAUNCH("dyn_tanh_close", (dyn_tanh_close_kernel<E, VEC, 1>), dim3(gx, a.rows), dim3(th), 0, s, (const E*)y, x, (E*)out_e, a);
    }
    return DLI_OK;
  }
  const size_t ld = ((size_t)a.d + 3) / 4 * 4, zl = moe_route_floats(ra->n_out, ra->groups);
  const int n_log = ra->n_out + (ra->sg_w ? 1 : 0);
  const size_t smem4 = kDytRouteRows * (ld + zl) * sizeof(float), smem1 = (ld + zl) * sizeof(float);
  DLI_CHECK_ARG(smem1 <= kDytRouteMaxSmem, "dli_dyn_tanh_close: width %d with %d router outputs needs %zu bytes of shared memory", a.d,
                ra->n_out, smem1);
  static PerDeviceOnce once1, once4;
  if (a.rows > kDytFewRows && smem4 <= kDytRouteMaxSmem) {
    DLI_ONCE_PER_DEVICE(once4, dev, DLI_CUDA_CALL(cudaFuncSetAttribute(dyn_tanh_close_route_kernel<E, VEC, kDytRouteRows>,
                                                                        cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kDytRouteMaxSmem)));
    int warps = (n_log + 1) / 2;                        // a warp per two logits in one round where that many fit
    warps = warps < 8 ? 8 : (warps > 16 ? 16 : warps);
    DLI_LAUNCH("dyn_tanh_close_route", (dyn_tanh_close_route_kernel<E, VEC, kDytRouteRows>), dim3((a.rows + kDytRouteRows - 1) / kDytRouteRows),
               dim3(32 * warps), smem4, s, (const E*)y, x, (E*)out_e, a, *ra);
  } else {
    DLI_ONCE_PER_DEVICE(once1, dev1, DLI_CUDA_CALL(cudaFuncSetAttribute(dyn_tanh_close_route_kernel<E, VEC, 1>,
                                                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kDytRouteMaxSmem)));
    int warps = n_log > 16 ? 32 : 16;                   // a warp per logit
    DLI_LAUNCH("dyn_tanh_close_route", (dyn_tanh_close_route_kernel<E, VEC, 1>), dim3(a.rows), dim3(32 * warps), smem1, s, (const E*)y, x,
               (E*)out_e, a, *ra);
  }
  return DLI_OK;
}

}  // namespace dli

using namespace dli;

extern "C" {

int dli_dyn_tanh_close(const void* y, const float* post_w, const float* post_b, float post_alpha, float mult, const float* add,
                       float* x, const float* next_w, const float* next_b, float next_alpha, float* out_f, void* out_e, int rows,
                       int d, int dt, const float* w_router, const float* logit_bias, const float* correction, float* r_wts,
                       float* r_idw, int32_t* r_sel_idx, float* r_sel_w, int n_out, int n_real, int top, int groups, int keep,
                       float wscale, int renorm, int score, const float* sg_w, float* sg, dli_stream_t stream) {
  DLI_CHECK_ARG(x && d > 0, "dli_dyn_tanh_close: null pointer or empty shape");
  DLI_CHECK_ARG(!y || (post_w && post_b), "dli_dyn_tanh_close: a sublayer result needs its map's weights");
  DLI_CHECK_ARG(y || add || next_w, "dli_dyn_tanh_close: nothing to do");
  DLI_CHECK_ARG((next_w == nullptr) == (next_b == nullptr), "dli_dyn_tanh_close: the map that follows needs w and b");
  DLI_CHECK_ARG(next_w ? (out_f || out_e || w_router) : !(out_f || out_e || w_router),
                "dli_dyn_tanh_close: outputs and router belong to the map that follows");
  DLI_CHECK_ARG(dt == 0 || dt == 1, "element type %d: 0 = bf16, 1 = float", dt);
  if (groups < 1) groups = 1;
  auto al = [](const void* p, uintptr_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  DLI_CHECK_ARG(!w_router || (r_wts && r_idw && r_sel_idx && r_sel_w && n_out > 0 && n_out <= 4096 && n_real >= 0 && n_real <= n_out &&
                              top > 0 && top <= n_out && (score == 0 || score == 1) && (!sg_w || sg) && al(w_router, 16) && al(sg_w, 16) &&
                              (groups == 1 || (n_out % groups == 0 && keep >= 1 && keep <= groups && keep * (n_out / groups) >= top))),
                "dli_dyn_tanh_close: the router needs its outputs; %d outputs (%d real), top %d, %d groups of which %d are kept, score %d",
                n_out, n_real, top, groups, keep, score);
  if (rows <= 0) return DLI_OK;
  DynTanhClose a{{post_w, post_b, post_alpha}, mult, add, {next_w, next_b, next_alpha}, out_f, rows, d};
  RouteArgs ra{w_router, correction, r_wts, r_idw, r_sel_idx, r_sel_w, n_out, n_real, top, groups, keep, wscale, renorm, logit_bias,
               score, sg_w, sg};
  const bool vec = d % 4 == 0 && al(x, 16) && al(y, dt == 0 ? 8 : 16) && al(post_w, 16) && al(post_b, 16) && al(add, 16) && al(next_w, 16) &&
                   al(next_b, 16) && al(out_f, 16) && al(out_e, dt == 0 ? 8 : 16);
  const RouteArgs* rp = w_router ? &ra : nullptr;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dt == 0) return vec ? launch_dyt<bf16, 4>(y, x, out_e, a, rp, s) : launch_dyt<bf16, 1>(y, x, out_e, a, rp, s);
  return vec ? launch_dyt<float, 4>(y, x, out_e, a, rp, s) : launch_dyt<float, 1>(y, x, out_e, a, rp, s);
}

}  // extern "C"
