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

// rows of whole 16-byte units
__device__ __forceinline__ float4 dyt_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 dyt_ld4(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void dyt_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void dyt_st4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

template <typename T>
__global__ void __launch_bounds__(256) dyt_v4_kernel(TpxDyt p) {
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const T* e = p.ids ? reinterpret_cast<const T*>(p.embed) + p.ids[row] * p.D : nullptr;
  const float* x = p.ids ? nullptr : p.x + row * p.D;
  float* xo = p.x_out ? p.x_out + row * p.D : nullptr;
  T* h = reinterpret_cast<T*>(p.h) + row * p.ldh;
  for (int d = threadIdx.x * 4; d < p.D; d += 1024) {
    float4 v;
    if (e) {
      v = dyt_ld4(e + d);
      v = make_float4(v.x * p.scale, v.y * p.scale, v.z * p.scale, v.w * p.scale);
    } else {
      v = dyt_ld4(x + d);
    }
    if (p.add) {
      const float4 a = dyt_ld4(p.add + d);
      v = make_float4(v.x + a.x, v.y + a.y, v.z + a.z, v.w + a.w);
    }
    if (xo) dyt_st4(xo + d, v);
    const float4 w = dyt_ld4(p.w + d), b = dyt_ld4(p.b + d);
    dyt_st4(h + d, make_float4(fmaf(tanhf(p.alpha * v.x), w.x, b.x), fmaf(tanhf(p.alpha * v.y), w.y, b.y), fmaf(tanhf(p.alpha * v.z), w.z, b.z),
                               fmaf(tanhf(p.alpha * v.w), w.w, b.w)));
  }
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_dyt(const TpxDyt* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "dyt: null argument block");
  TPX_REQUIRE(a->n >= 0 && a->n < (1ll << 31) && a->D > 0 && a->D < (1 << 20) && a->ldh >= a->D, TPX_ERR_ARG, "dyt: bad shape");
  if (a->n == 0) return TPX_OK;
  TPX_REQUIRE((a->ids ? a->embed != nullptr : a->x != nullptr) && a->w && a->b && a->h, TPX_ERR_ARG, "dyt: null pointer");
  const uintptr_t all = (uintptr_t)a->embed | (uintptr_t)a->x | (uintptr_t)a->add | (uintptr_t)a->w | (uintptr_t)a->b | (uintptr_t)a->x_out | (uintptr_t)a->h;
  const bool v4 = a->D % 4 == 0 && a->ldh == a->D && (all & 15) == 0;
  void (*k)(TpxDyt) = v4 ? (a->f32 ? dyt_v4_kernel<float> : dyt_v4_kernel<__nv_bfloat16>) : (a->f32 ? dyt_kernel<float> : dyt_kernel<__nv_bfloat16>);
  TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)a->n), dim3(256), 0, (cudaStream_t)stream, *a));
  return TPX_OK;
}
