// Helpers shared by the hybrid decoder's kernels: element types, reductions, activations.
#pragma once
#include "tpx_common.cuh"
#include "../../include/tpx_hybrid.h"

namespace tpx {

template <typename T>
__device__ __forceinline__ float hy_ld(const T* p);
template <>
__device__ __forceinline__ float hy_ld<float>(const float* p) { return *p; }
template <>
__device__ __forceinline__ float hy_ld<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T>
__device__ __forceinline__ void hy_st(T* p, float v);
template <>
__device__ __forceinline__ void hy_st<float>(float* p, float v) { *p = v; }
template <>
__device__ __forceinline__ void hy_st<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float hy_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Sum over a block of at most 1024 threads; every thread receives it. red: 32 floats of shared memory, free again on return.
__device__ __forceinline__ float hy_block_sum(float v, float* red) {
  v = hy_warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const int nw = (blockDim.x + 31) >> 5;
  float s = 0.0f;
  for (int i = 0; i < nw; i++) s += red[i];
  __syncthreads();
  return s;
}

__device__ __forceinline__ float hy_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }

__device__ __forceinline__ float hy_act(float v, int act, float a0, float a1) {
  switch (act) {
    case TPX_ACT_TANH: return tanhf(v);
    case TPX_ACT_XIELU: return v > 0.0f ? fmaf(a0 * v, v, 0.5f * v) : fmaf(a1, expm1f(v) - v, 0.5f * v);
    default: return apply_act(v, act);
  }
}

// one unit of the clamped gated feed-forward
__device__ __forceinline__ float hy_clamped_glu(float g, float u, float limit) {
  g = fminf(g, limit);
  return g * hy_sigmoid(1.702f * g) * (fminf(fmaxf(u, -limit), limit) + 1.0f);
}

// bf16 decoding of latent attention (tpx_latent_dec.cu)
bool latent_absorb_mma_serves(const TpxLatentAbsorb& a);
int latent_absorb_mma(const TpxLatentAbsorb& a, cudaStream_t st);
bool latent_value_mma_serves(const TpxLatentValue& a);
int latent_value_mma(const TpxLatentValue& a, cudaStream_t st);
bool latent_decode_serves(const TpxLatentAttn& a);
int latent_decode(const TpxLatentAttn& a, cudaStream_t st);

// the bf16 operands of tpx_linear on the tcgen05 kernel (tpx_linear_bf16.cu)
int linear_tc_ex(const TpxLinear& a, cudaStream_t st);

// as above for a bf16 result: special-function exponential, approximate quotient
__device__ __forceinline__ float hy_clamped_glu_fast(float g, float u, float limit) {
  g = fminf(g, limit);
  return __fdividef(g, 1.0f + __expf(-1.702f * g)) * (fminf(fmaxf(u, -limit), limit) + 1.0f);
}

// chunked differential attention in bf16: several tokens (tpx_diff_tc.cu), one token, append included (tpx_diff_dec.cu)
bool diff_prefill_serves(int64_t dim, int64_t vdim, float softcap);
int diff_prefill(const TpxDiffAttn& a, cudaStream_t st);
bool diff_decode_serves(const TpxDiffAttn& a);
int diff_decode(const TpxDiffAttn& a, cudaStream_t st);

}  // namespace tpx
