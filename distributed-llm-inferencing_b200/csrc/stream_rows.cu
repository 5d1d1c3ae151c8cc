// Row-wise pieces of layers with SEVERAL RESIDUAL STREAMS (hyper-connections) on a ragged step.  Instead of one row x
// there are S rows x_0 .. x_(S-1), fp32.  A sublayer reads u = sum_s in[s] x_s, and with y = sublayer(norm(u) * w) all
// streams are replaced at once:  x_t <- sum_s mix[s, t] x_s + out[t] y   (mix indexed [from, to]).
//
// dli_streams_close does everything between two projections in one pass over the row: the new streams from the old
// ones and the sublayer's result, the NEXT sublayer's u (or, with no weights given, the sum of the streams, which the
// model's last norm reads), its RMS norm as fp32 and / or element-type rows and, where a mixture of experts follows,
// the router on the normed row.  Without a sublayer result it only reads (the first sublayer of a model).
#include "common.cuh"
#include "moe_route.cuh"

namespace dli {

struct StreamsClose {
  float* x;               // stream s of row r at x + s * xs_stride + r * d
  size_t xs_stride;
  const float* mix;       // [S, S] from, to
  const float* outw;      // [S]
  const float* in_next;   // [S] or NULL (ones)
  const float* w_next;    // [d] or NULL: no norm
  float* out_f;           // [rows, d] or NULL
  float eps;
  int d;
  int has_route;
  RouteArgs route;
};

template <int VEC> struct Vecf { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Vecf<VEC> sr_ld(const float* p) {
  Vecf<VEC> r;
  if constexpr (VEC == 4) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    r.v[0] = u.x; r.v[1] = u.y; r.v[2] = u.z; r.v[3] = u.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int VEC> __device__ __forceinline__ Vecf<VEC> sr_ld(const bf16* p) {
  Vecf<VEC> r;
  if constexpr (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    r.v[0] = bf_lo(u.x); r.v[1] = bf_hi(u.x); r.v[2] = bf_lo(u.y); r.v[3] = bf_hi(u.y);
  } else {
    r.v[0] = __bfloat162float(*p);
  }
  return r;
}
template <int VEC> __device__ __forceinline__ void sr_st(float* p, const Vecf<VEC>& r) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int VEC> __device__ __forceinline__ void sr_st(bf16* p, const Vecf<VEC>& r) {
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(r.v[0], r.v[1]), pack_bf16(r.v[2], r.v[3]));
  else *p = __float2bfloat16_rn(r.v[0]);
}

// One CTA per row.  Pass 1: new streams, u (kept in shared memory) and its sum of squares; pass 2: the norm.
// Dynamic shared memory: [d] u, then the router's scratch.
template <typename E, int VEC, int S>
__global__ void __launch_bounds__(1024)
streams_close_kernel(const E* __restrict__ y, E* __restrict__ out_e, StreamsClose a) {
  extern __shared__ __align__(16) float ubuf[];
  __shared__ float red[32];
  float mix[S][S], ow[S], iw[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {  // weights: not written by any kernel, read before the wait
    iw[s] = a.in_next ? a.in_next[s] : 1.f;
    ow[s] = y ? a.outw[s] : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = y ? a.mix[s * S + t] : 0.f;
  }
  pdl_wait();
  pdl_trigger();
  const int row = blockIdx.x, d = a.d;
  const size_t o = (size_t)row * d;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < d; c += blockDim.x * VEC) {
    Vecf<VEC> x[S], u;
#pragma unroll
    for (int s = 0; s < S; ++s) x[s] = sr_ld<VEC>(a.x + s * a.xs_stride + o + c);
    if (y) {
      const Vecf<VEC> yv = sr_ld<VEC>(y + o + c);
      Vecf<VEC> n[S];
#pragma unroll
      for (int t = 0; t < S; ++t) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          float v = ow[t] * yv.v[i];
#pragma unroll
          for (int s = 0; s < S; ++s) v = fmaf(mix[s][t], x[s].v[i], v);
          n[t].v[i] = v;
        }
        sr_st<VEC>(a.x + t * a.xs_stride + o + c, n[t]);
      }
#pragma unroll
      for (int s = 0; s < S; ++s) x[s] = n[s];
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      float v = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) v = fmaf(iw[s], x[s].v[i], v);
      u.v[i] = v;
      ss = fmaf(v, v, ss);
    }
    if (a.w_next) sr_st<VEC>(ubuf + c, u);
  }
  if (!a.w_next) return;
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) ss += red[i];
  const float r = 1.f / sqrtf(ss / d + a.eps);
  for (int c = threadIdx.x * VEC; c < d; c += blockDim.x * VEC) {
    Vecf<VEC> h = sr_ld<VEC>(ubuf + c);
    const Vecf<VEC> w = sr_ld<VEC>(a.w_next + c);
#pragma unroll
    for (int i = 0; i < VEC; ++i) h.v[i] = h.v[i] * r * w.v[i];
    if (a.out_f) sr_st<VEC>(a.out_f + o + c, h);
    if (out_e) sr_st<VEC>(out_e + o + c, h);
    if (a.has_route) sr_st<VEC>(ubuf + c, h);
  }
  if (a.has_route) {
    __syncthreads();  // the normed row in shared memory is complete
    moe_route_row(ubuf, d, row, a.route, ubuf + ((d + 3) / 4) * 4);
  }
}

template <typename E, int S>
static int launch_streams(const void* y, void* out_e, const StreamsClose& a, int rows, bool vec, size_t smem, int th, cudaStream_t s) {
  if (vec) DLI_LAUNCH("streams_close", (streams_close_kernel<E, 4, S>), dim3(rows), dim3(th), smem, s, (const E*)y, (E*)out_e, a);
  else DLI_LAUNCH("streams_close", (streams_close_kernel<E, 1, S>), dim3(rows), dim3(th), smem, s, (const E*)y, (E*)out_e, a);
  return DLI_OK;
}

template <typename E>
static int dispatch_streams(const void* y, void* out_e, const StreamsClose& a, int S, int rows, bool vec, size_t smem, int th, cudaStream_t s) {
  switch (S) {
    case 1: return launch_streams<E, 1>(y, out_e, a, rows, vec, smem, th, s);
    case 2: return launch_streams<E, 2>(y, out_e, a, rows, vec, smem, th, s);
    case 3: return launch_streams<E, 3>(y, out_e, a, rows, vec, smem, th, s);
    case 4: return launch_streams<E, 4>(y, out_e, a, rows, vec, smem, th, s);
    case 5: return launch_streams<E, 5>(y, out_e, a, rows, vec, smem, th, s);
    case 6: return launch_streams<E, 6>(y, out_e, a, rows, vec, smem, th, s);
    case 7: return launch_streams<E, 7>(y, out_e, a, rows, vec, smem, th, s);
    default: return launch_streams<E, 8>(y, out_e, a, rows, vec, smem, th, s);
  }
}

}  // namespace dli

using namespace dli;

extern "C" {

int dli_streams_close(const void* y, float* x, size_t xs_stride, int n_streams, const float* mix, const float* outw,
                      const float* in_next, const float* w_next, float* out_f, void* out_e, int rows, int d, float eps, int dt,
                      const float* w_router, const float* logit_bias, const float* correction, float* r_wts, float* r_idw,
                      int32_t* r_sel_idx, float* r_sel_w, int n_out, int n_real, int top, int groups, int keep, float wscale,
                      int renorm, dli_stream_t stream) {
  DLI_CHECK_ARG(x && d > 0 && n_streams >= 1 && n_streams <= 8 && (n_streams == 1 || xs_stride >= (size_t)rows * d),
                "dli_streams_close: null pointer, empty shape or %d streams (1..8)", n_streams);
  DLI_CHECK_ARG(!y || (mix && outw), "dli_streams_close: a sublayer result needs the mixing and output weights");
  DLI_CHECK_ARG(y || w_next, "dli_streams_close: nothing to do");
  DLI_CHECK_ARG(!w_next || out_f || out_e || w_router, "dli_streams_close: the norm has no output");
  DLI_CHECK_ARG(dt == 0 || dt == 1, "element type %d: 0 = bf16, 1 = float", dt);
  if (groups < 1) groups = 1;
  DLI_CHECK_ARG(!w_router || (w_next && r_wts && r_idw && r_sel_idx && r_sel_w && n_out > 0 && n_out <= 4096 && n_real >= 0 &&
                              n_real <= n_out && top > 0 && top <= n_out && (reinterpret_cast<uintptr_t>(w_router) & 15u) == 0 &&
                              (groups == 1 || (n_out % groups == 0 && keep >= 1 && keep <= groups && keep * (n_out / groups) >= top))),
                "dli_streams_close: the router needs the norm and its outputs; %d outputs (%d real), top %d, %d groups of which %d are kept",
                n_out, n_real, top, groups, keep);
  const size_t smem = sizeof(float) * ((w_next ? ((size_t)d + 3) / 4 * 4 : 0) + (w_router ? (size_t)moe_route_floats(n_out, groups) : 0));
  DLI_CHECK_ARG(smem <= 48 * 1024, "dli_streams_close: width %d needs %zu bytes of shared memory", d, smem);
  if (rows <= 0) return DLI_OK;
  StreamsClose a{x, xs_stride, mix, outw, in_next, w_next, out_f, eps, d, w_router ? 1 : 0,
                 RouteArgs{w_router, correction, r_wts, r_idw, r_sel_idx, r_sel_w, n_out, n_real, top, groups, keep, wscale, renorm,
                           logit_bias}};
  auto al = [](const void* p, uintptr_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const bool vec = d % 4 == 0 && al(x, 16) && xs_stride % 4 == 0 && al(y, dt == 0 ? 8 : 16) && al(w_next, 16) && al(out_f, 16) &&
                   al(out_e, dt == 0 ? 8 : 16);
  const int per = vec ? 4 : 1;
  int th = (rows <= 64 && d >= 2048 * per) ? 1024 : (d >= 256 * per ? 256 : 128);
  if (w_router && th < (rows <= 64 ? 512 : 256)) th = rows <= 64 ? 512 : 256;  // a warp per router output
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dt == 0 ? dispatch_streams<bf16>(y, out_e, a, n_streams, rows, vec, smem, th, s)
                 : dispatch_streams<float>(y, out_e, a, n_streams, rows, vec, smem, th, s);
}

}  // extern "C"
