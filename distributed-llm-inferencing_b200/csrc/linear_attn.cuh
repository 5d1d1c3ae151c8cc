// Shared by the CUDA-core and the tensor-core forms of linear attention (linear_attn.cu, linear_attn_tc.cu).
#pragma once
#include "common.cuh"

namespace dli {

template <typename E> __device__ __forceinline__ float l_to_f(E v);
template <> __device__ __forceinline__ float l_to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float l_to_f<bf16>(bf16 v) { return __bfloat162float(v); }

struct LinAttn {
  const int32_t* ent;
  int H, D, V;
  int ldp, q_off, k_off, v_off;
  int silu;                 // SiLU on q, k and v
  float q_scale, k_scale;
  const float* cos_t;       // [positions, rd/2]
  const float* sin_t;
  int rd;
  const float* log_decay;   // [H]: log of the fixed decay, or NULL:
  int a_off, rank;          // columns of a_t
  const float* a2;          // [H*D, rank]
  const float* a2_b;        // [H*D]
  float inv_tau;
};

// one prepared entry of q or k: column `base + i` of the projection row, i within the head
template <typename E>
__device__ __forceinline__ float la_qk(const E* pr, int base, int i, const LinAttn& a, int pos, float scale) {
  float u = l_to_f(pr[base + i]);
  if (a.silu) u = silu_f(u);
  if (i < a.rd) {
    const int half = a.rd >> 1, j = i < half ? i : i - half;
    float p = l_to_f(pr[base + (i < half ? i + half : j)]);
    if (a.silu) p = silu_f(p);
    const float c = a.cos_t[(size_t)pos * half + j], s = a.sin_t[(size_t)pos * half + j];
    u = i < half ? u * c - p * s : u * c + p * s;
  }
  return u * scale;
}

constexpr int kLaTile = 64;   // rows per tile of the tile-parallel forms

// linear_attn_tc.cu: the tiles' state contributions and read-outs on the tensor cores (bf16 projection rows).  row_scr: the
// rows' log decays [rows, H*D], or, with a fixed decay, scratch of rows * (2HD + HV) floats that local fills and out reads.
bool linattn_tc_supported(const LinAttn& a);
int linattn_tc_local(const void* proj, float* row_scr, const LinAttn& a, int rows, const int32_t* tiles, int n_tiles, float* scr_u,
                     float* scr_w, cudaStream_t s);
int linattn_tc_out(const void* proj, float* row_scr, float* o, const LinAttn& a, int rows, const int32_t* tiles, int n_tiles,
                   const float* scr_u, cudaStream_t s);

}  // namespace dli
