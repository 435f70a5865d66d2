// The residual stream of a decoder whose norm is a Dynamic Tanh, h = tanh(alpha x) w + b, element by element: the start of the
// stream (embedding rows, scaled) or a bare norm. Behind a linear both the sum and the norm are the linear's epilogue.
#include "tpx_hybrid.cuh"

namespace tpx {

template <typename T>
__global__ void __launch_bounds__(256) dyt_kernel(TpxDyt p) {
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x, D = p.D;
  const T* e = p.ids ? reinterpret_cast<const T*>(p.embed) + p.ids[row] * D : nullptr;
  const float* x = p.ids ? nullptr : p.x + row * D;
  float* xo = p.x_out ? p.x_out + row * D : nullptr;
  T* h = reinterpret_cast<T*>(p.h) + row * p.ldh;
  for (int64_t d = threadIdx.x; d < p.ldh; d += 256) {
    float r = 0.0f;
    if (d < D) {
      float v = e ? hy_ld(e + d) * p.scale : x[d];
      if (p.add) v += p.add[d];
      if (xo) xo[d] = v;
      r = fmaf(tanhf(p.alpha * v), p.w[d], p.b[d]);
    }
    hy_st(h + d, r);
  }
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_dyt(const TpxDyt* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "dyt: null argument block");
  TPX_REQUIRE(a->n >= 0 && a->n < (1ll << 31) && a->D > 0 && a->D < (1 << 20) && a->ldh >= a->D, TPX_ERR_ARG, "dyt: bad shape");
  if (a->n == 0) return TPX_OK;
  TPX_REQUIRE((a->ids ? a->embed != nullptr : a->x != nullptr) && a->w && a->b && a->h, TPX_ERR_ARG, "dyt: null pointer");
  void (*k)(TpxDyt) = a->f32 ? dyt_kernel<float> : dyt_kernel<__nv_bfloat16>;
  TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)a->n), dim3(256), 0, (cudaStream_t)stream, *a));
  return TPX_OK;
}
