// Sub-layer boundary of a post-norm decoder: x <- norm(alpha x + y) in 32-bit, fused with the causal per-channel input
// convolution of the next sub-layer, h = x + conv(x); the end of the stream (last norm, final norm, rows wanted only); and
// the greedy pick over fp32 logits.
//
// Many tokens: a CTA owns 16 consecutive tokens of one sequence and the taps - 1 before them. A warp per token first
// computes the inverse root mean squares, then every thread walks its channels through the tokens with the convolution's
// history in registers. One token per sequence: a CTA per sequence, the history in the layer's state.
#include "tpx_hybrid.cuh"

namespace tpx {

constexpr int kPncThreads = 256, kPncTokens = 16, kPncMaxTaps = 64;

template <typename T>
struct PncParams {
  const int64_t* ids;
  const T* embed;
  const float *x, *y, *w, *conv;
  float* state;
  const int *start, *dev_len;
  float* x_out;
  T* h;
  int B, S, D, ldh, past, taps;
  float alpha, eps;
};

// the sum alpha x + y of row `row`, channel d; at the start of the stream the embedding of token `id`
template <typename T>
__device__ __forceinline__ float pnc_sum(const PncParams<T>& p, int64_t row, int64_t id, int d) {
  return p.ids ? hy_ld(p.embed + id * p.D + d) : fmaf(p.alpha, p.x[row * p.D + d], p.y[row * p.D + d]);
}

template <typename T>
__global__ void __launch_bounds__(kPncThreads) pnc_token_kernel(PncParams<T> p) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x;
  const int64_t row = b, id = p.ids ? p.ids[b] : 0;
  const int t = p.dev_len ? *p.dev_len : p.past;
  const bool pad = p.start && t < p.start[b];
  float inv = 1.0f;
  if (!p.ids) {
    float ss = 0.0f;
    for (int d = threadIdx.x; d < p.D; d += kPncThreads) {
      const float z = pnc_sum(p, row, id, d);
      ss = fmaf(z, z, ss);
    }
    inv = 1.0f / sqrtf(hy_block_sum(ss, red) / (float)p.D + p.eps);
  }
  for (int d = threadIdx.x; d < p.D; d += kPncThreads) {
    float v = pnc_sum(p, row, id, d);
    if (!p.ids) v = v * inv * (1.0f + p.w[d]);
    if (pad) v = 0.0f;
    if (p.conv) {
      float c = p.conv[(int64_t)(p.taps - 1) * p.D + d] * v;
      float* st = p.state + ((int64_t)b * (p.taps - 1)) * p.D + d;
      for (int j = 0; j < p.taps - 1; j++) {
        const float o = st[(int64_t)j * p.D];
        c = fmaf(p.conv[(int64_t)j * p.D + d], o, c);
        if (j > 0) st[(int64_t)(j - 1) * p.D] = o;
      }
      if (p.taps > 1) st[(int64_t)(p.taps - 2) * p.D] = v;
      hy_st(p.h + row * p.ldh + d, v + c);
    }
    p.x_out[row * p.D + d] = v;
  }
  if (p.conv)
    for (int d = p.D + threadIdx.x; d < p.ldh; d += kPncThreads) hy_st(p.h + row * p.ldh + d, 0.0f);
}

// Any width and number of taps; a tap's earlier token is recomputed from the sum.
template <typename T>
__global__ void __launch_bounds__(kPncThreads) pnc_tokens_kernel(PncParams<T> p) {
  __shared__ float s_inv[kPncTokens + kPncMaxTaps];  // < 0: a row that counts as zero
  __shared__ int64_t s_id[kPncTokens + kPncMaxTaps];
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, s0 = blockIdx.x * kPncTokens;
  const int s1 = min(p.S, s0 + kPncTokens);
  const int halo = p.conv ? p.taps - 1 : 0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pads = p.start ? p.start[b] - p.past : 0;  // tokens s < pads of this call are padding
  const int64_t row0 = (int64_t)b * p.S;
  for (int i = warp; i < s1 - s0 + halo; i += kPncThreads / 32) {
    const int s = s0 - halo + i;
    float inv = 1.0f;
    if (s < pads) inv = -1.0f;
    else if (s >= 0 && !p.ids) {
      float ss = 0.0f;
      for (int d = lane; d < p.D; d += 32) {
        const float z = pnc_sum(p, row0 + s, 0, d);
        ss = fmaf(z, z, ss);
      }
      inv = 1.0f / sqrtf(hy_warp_sum(ss) / (float)p.D + p.eps);
    }
    if (lane == 0) {
      s_inv[i] = inv;
      s_id[i] = (p.ids && s >= 0) ? p.ids[row0 + s] : 0;
    }
  }
  __syncthreads();
  for (int d = threadIdx.x; d < p.D; d += kPncThreads) {
    const float g = p.ids ? 1.0f : 1.0f + p.w[d];
    auto value = [&](int s) -> float {  // the normed stream at token s of this call, s < 0: from the state
      const int i = s - s0 + halo;
      if (s < 0) return p.state[((int64_t)b * (p.taps - 1) + s + p.taps - 1) * p.D + d];
      if (s_inv[i] < 0.0f) return 0.0f;
      return pnc_sum(p, row0 + s, s_id[i], d) * s_inv[i] * g;
    };
    for (int s = s0; s < s1; s++) {
      const float v = value(s);
      p.x_out[(row0 + s) * p.D + d] = v;
      if (!p.conv) continue;
      float c = v;
      for (int j = 0; j < p.taps; j++) c = fmaf(p.conv[(int64_t)j * p.D + d], j == p.taps - 1 ? v : value(s - (p.taps - 1) + j), c);
      hy_st(p.h + (row0 + s) * p.ldh + d, c);
    }
  }
  if (p.conv)
    for (int s = s0; s < s1; s++)
      for (int d = p.D + threadIdx.x; d < p.ldh; d += kPncThreads) hy_st(p.h + (row0 + s) * p.ldh + d, 0.0f);
}

// ---------------------------------------------------------------- whole float4 vectors, up to four taps
__device__ __forceinline__ float4 pnc_fma4(float a, float4 x, float4 y) {
  return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}
__device__ __forceinline__ float4 pnc_fma4(float4 a, float4 x, float4 y) {
  return make_float4(fmaf(a.x, x.x, y.x), fmaf(a.y, x.y, y.y), fmaf(a.z, x.z, y.z), fmaf(a.w, x.w, y.w));
}
__device__ __forceinline__ float pnc_dot4(float4 a) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, a.w * a.w))); }
__device__ __forceinline__ float4 pnc_scale4(float4 z, float inv, float4 w) {
  return make_float4(z.x * inv * (1.0f + w.x), z.y * inv * (1.0f + w.y), z.z * inv * (1.0f + w.z), z.w * inv * (1.0f + w.w));
}
__device__ __forceinline__ float4 pnc_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 pnc_ld4(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void pnc_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void pnc_st4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

constexpr int kPncV4Threads = 512, kPncV4 = 4;  // one token: up to 4 vectors per thread, rows up to 8192 elements

// One token per sequence, everything in registers; the weights are fetched before the earlier kernels are waited for.
template <typename T, int TAPS, int NV>
__global__ void __launch_bounds__(kPncV4Threads) pnc_token_v4_kernel(PncParams<T> p) {
  __shared__ float red[32];
  pdl_trigger();
  const int b = blockIdx.x, nv = p.D / 4;
  float4 w[NV], cw[NV][TAPS];
#pragma unroll
  for (int q = 0; q < NV; q++) {
    const int i = threadIdx.x + q * kPncV4Threads;
    if (i < nv) {
      w[q] = p.ids ? make_float4(0, 0, 0, 0) : __ldg(reinterpret_cast<const float4*>(p.w) + i);
#pragma unroll
      for (int j = 0; j < TAPS; j++) cw[q][j] = __ldg(reinterpret_cast<const float4*>(p.conv + (int64_t)j * p.D) + i);
    }
  }
  pdl_wait();
  const int t = p.dev_len ? *p.dev_len : p.past;
  const bool pad = p.start && t < p.start[b];
  float* state = p.state + (int64_t)b * (TAPS - 1) * p.D;
  float4 z[NV], hist[NV][TAPS];
  float ss = 0.0f;
#pragma unroll
  for (int q = 0; q < NV; q++) {
    const int i = threadIdx.x + q * kPncV4Threads;
    z[q] = make_float4(0, 0, 0, 0);
    if (i < nv) {
      if (p.ids) z[q] = pnc_ld4(p.embed + p.ids[b] * p.D + i * 4);
      else z[q] = pnc_fma4(p.alpha, pnc_ld4(p.x + (int64_t)b * p.D + i * 4), pnc_ld4(p.y + (int64_t)b * p.D + i * 4));
#pragma unroll
      for (int j = 0; j < TAPS - 1; j++) hist[q][j] = pnc_ld4(state + (int64_t)j * p.D + i * 4);
    }
    ss += pnc_dot4(z[q]);
  }
  const float inv = p.ids ? 1.0f : 1.0f / sqrtf(hy_block_sum(ss, red) / (float)p.D + p.eps);
#pragma unroll
  for (int q = 0; q < NV; q++) {
    const int i = threadIdx.x + q * kPncV4Threads;
    if (i < nv) {
      const float4 v = pad ? make_float4(0, 0, 0, 0) : pnc_scale4(z[q], inv, w[q]);
      hist[q][TAPS - 1] = v;
      float4 c = v;
#pragma unroll
      for (int j = 0; j < TAPS; j++) c = pnc_fma4(cw[q][j], hist[q][j], c);
#pragma unroll
      for (int j = 0; j < TAPS - 1; j++) pnc_st4(state + (int64_t)j * p.D + i * 4, hist[q][j + 1]);
      pnc_st4(p.h + (int64_t)b * p.ldh + i * 4, c);
      pnc_st4(p.x_out + (int64_t)b * p.D + i * 4, v);
    }
  }
  for (int d = p.D + threadIdx.x; d < p.ldh; d += kPncV4Threads) hy_st(p.h + (int64_t)b * p.ldh + d, 0.0f);
}

// Many tokens, as pnc_tokens_kernel with the history in registers.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kPncThreads) pnc_tokens_v4_kernel(PncParams<T> p) {
  constexpr int HALO = TAPS - 1, N = kPncTokens + HALO;
  __shared__ float s_inv[N];  // < 0: a row that counts as zero
  __shared__ int64_t s_id[N];
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, s0 = blockIdx.x * kPncTokens, nv = p.D / 4;
  const int n = min(p.S - s0, kPncTokens);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pads = p.start ? p.start[b] - p.past : 0;
  const int64_t row0 = (int64_t)b * p.S + s0;
  const float* __restrict__ x = p.ids ? nullptr : p.x + row0 * p.D;
  const float* __restrict__ y = p.ids ? nullptr : p.y + row0 * p.D;
  float* __restrict__ xo = p.x_out + row0 * p.D;
  T* __restrict__ h = p.h + row0 * p.ldh;
  for (int i = warp; i < n + HALO; i += kPncThreads / 32) {
    const int s = i - HALO;  // relative to s0
    float inv = 1.0f;
    if (s0 + s < pads) inv = -1.0f;
    else if (s0 + s >= 0 && !p.ids) {
      float ss = 0.0f;
#pragma unroll 4
      for (int v = lane; v < nv; v += 32) ss += pnc_dot4(pnc_fma4(p.alpha, pnc_ld4(x + (int64_t)s * p.D + v * 4), pnc_ld4(y + (int64_t)s * p.D + v * 4)));
      inv = 1.0f / sqrtf(hy_warp_sum(ss) / (float)p.D + p.eps);
    }
    if (lane == 0) {
      s_inv[i] = inv;
      s_id[i] = (p.ids && s0 + s >= 0) ? p.ids[row0 + s] : 0;
    }
  }
  __syncthreads();
  for (int v = threadIdx.x; v < nv; v += kPncThreads) {
    const float4 w = p.ids ? make_float4(0, 0, 0, 0) : __ldg(reinterpret_cast<const float4*>(p.w) + v);
    auto raw = [&](int s) -> float4 {  // s relative to s0, in the call
      if (p.ids) return pnc_ld4(p.embed + s_id[s + HALO] * p.D + v * 4);
      return pnc_fma4(p.alpha, pnc_ld4(x + (int64_t)s * p.D + v * 4), pnc_ld4(y + (int64_t)s * p.D + v * 4));
    };
    auto norm = [&](float4 z, int s) -> float4 {
      const float inv = s_inv[s + HALO];
      return inv < 0.0f ? make_float4(0, 0, 0, 0) : pnc_scale4(z, inv, w);
    };
    float4 hist[TAPS], cw[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; j++) cw[j] = __ldg(reinterpret_cast<const float4*>(p.conv + (int64_t)j * p.D) + v);
#pragma unroll
    for (int j = 0; j < HALO; j++) {
      const int s = j - HALO;
      hist[j] = s0 + s < 0 ? pnc_ld4(p.state + ((int64_t)b * HALO + s0 + s + HALO) * p.D + v * 4) : norm(raw(s), s);
    }
    for (int s = 0; s < n; s += 4) {
      float4 z[4];
#pragma unroll
      for (int u = 0; u < 4; u++) z[u] = raw(min(s + u, n - 1));
#pragma unroll
      for (int u = 0; u < 4; u++) {
        if (s + u < n) {
          hist[TAPS - 1] = norm(z[u], s + u);
          float4 c = hist[TAPS - 1];
#pragma unroll
          for (int j = 0; j < TAPS; j++) c = pnc_fma4(cw[j], hist[j], c);
          pnc_st4(xo + (int64_t)(s + u) * p.D + v * 4, hist[TAPS - 1]);
          pnc_st4(h + (int64_t)(s + u) * p.ldh + v * 4, c);
#pragma unroll
          for (int j = 0; j < HALO; j++) hist[j] = hist[j + 1];
        }
      }
    }
  }
  for (int s = 0; s < n; s++)
    for (int d = p.D + threadIdx.x; d < p.ldh; d += kPncThreads) hy_st(h + (int64_t)s * p.ldh + d, 0.0f);
}

template <typename T, int TAPS>
static int pnc_run_v4(const PncParams<T>& p, cudaStream_t st) {
  if (p.S == 1) {
    const int nv = (p.D / 4 + kPncV4Threads - 1) / kPncV4Threads;
    void (*k)(PncParams<T>) = nv <= 1 ? pnc_token_v4_kernel<T, TAPS, 1> : nv <= 2 ? pnc_token_v4_kernel<T, TAPS, 2> : pnc_token_v4_kernel<T, TAPS, 4>;
    TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)p.B), dim3(kPncV4Threads), 0, st, p));
  } else {
    TPX_CUDA_OK(launch_pdl(pnc_tokens_v4_kernel<T, TAPS>, dim3((unsigned)((p.S + kPncTokens - 1) / kPncTokens), (unsigned)p.B), dim3(kPncThreads), 0, st, p));
  }
  return TPX_OK;
}

// after several tokens: the last taps - 1 inputs of every channel, x_out [B][S][D] holding the new ones
__global__ void __launch_bounds__(256) pnc_state_kernel(const float* __restrict__ x, float* __restrict__ state, int S, int D, int keep) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, d = blockIdx.x * 256 + threadIdx.x;
  if (d >= D) return;
  float* st = state + (int64_t)b * keep * D + d;
  for (int j = 0; j < keep; j++) {  // ascending: an old entry is read (j + S) before it is overwritten
    const int s = S - keep + j;
    st[(int64_t)j * D] = s < 0 ? st[(int64_t)(j + S) * D] : x[((int64_t)b * S + s) * D + d];
  }
}

template <typename T>
__global__ void __launch_bounds__(256) pnc_final_kernel(const float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w,
                                                        const float* __restrict__ wf, const int64_t* __restrict__ rows, T* __restrict__ out,
                                                        int D, int ldo, float alpha, float eps) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = rows[blockIdx.x];
  x += row * D;
  y += row * D;
  out += (int64_t)blockIdx.x * ldo;
  float ss = 0.0f;
  for (int d = threadIdx.x; d < D; d += 256) {
    const float z = fmaf(alpha, x[d], y[d]);
    ss = fmaf(z, z, ss);
  }
  const float inv = 1.0f / sqrtf(hy_block_sum(ss, red) / (float)D + eps);
  ss = 0.0f;
  for (int d = threadIdx.x; d < D; d += 256) {
    const float z = fmaf(alpha, x[d], y[d]) * inv * (1.0f + w[d]);
    ss = fmaf(z, z, ss);
  }
  const float inv2 = 1.0f / sqrtf(hy_block_sum(ss, red) / (float)D + eps);
  for (int d = threadIdx.x; d < D; d += 256) hy_st(out + d, fmaf(alpha, x[d], y[d]) * inv * (1.0f + w[d]) * inv2 * (1.0f + wf[d]));
  for (int d = D + threadIdx.x; d < ldo; d += 256) hy_st(out + d, 0.0f);
}

__global__ void __launch_bounds__(256) argmax_f32_kernel(const float* __restrict__ x, long long n, long long* __restrict__ out) {
  __shared__ float sv[8];
  __shared__ long long si[8];
  pdl_trigger();
  pdl_wait();
  x += (long long)blockIdx.x * n;
  float bv = -INFINITY;
  long long bi = 0;
  auto take = [&](float v, long long i) {
    const bool vn = v != v, bn = bv != bv;  // a NaN counts as the largest, as in torch.argmax
    if (vn != bn ? vn : (!vn && v != bv) ? v > bv : i < bi) { bv = v; bi = i; }
  };
  bool any = false;
  for (long long i = threadIdx.x; i < n; i += 256) {
    if (!any) { bv = x[i]; bi = i; any = true; }
    else take(x[i], i);
  }
  if (!any) bi = 0x7fffffffffffffffLL;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float v = __shfl_xor_sync(0xffffffffu, bv, o);
    const long long i = __shfl_xor_sync(0xffffffffu, bi, o);
    take(v, i);
  }
  if ((threadIdx.x & 31) == 0) { sv[threadIdx.x >> 5] = bv; si[threadIdx.x >> 5] = bi; }
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int i = 1; i < 8; i++) take(sv[i], si[i]);
    out[blockIdx.x] = bi;
  }
}

template <typename T>
static int pnc_run(const TpxPostnormConv& a, cudaStream_t st) {
  PncParams<T> p = {a.ids, (const T*)a.embed, a.x, a.y, a.w, a.conv, a.state, a.start, a.dev_len, a.x_out, (T*)a.h,
                    (int)a.B, (int)a.S, (int)a.D, (int)a.ldh, (int)a.past, a.taps, a.alpha, a.eps};
  auto aligned = [](const void* q) { return ((uintptr_t)q & 15) == 0; };
  const bool v4 = a.conv && a.D % 4 == 0 && a.ldh % 4 == 0 && a.taps <= 4 && (a.S > 1 || a.D <= kPncV4Threads * kPncV4 * 4) && aligned(a.x) && aligned(a.y) &&
                  aligned(a.w) && aligned(a.conv) && aligned(a.state) && aligned(a.x_out) && aligned(a.h) && aligned(a.embed);
  if (v4) {
    const int rc = a.taps == 1 ? pnc_run_v4<T, 1>(p, st) : a.taps == 2 ? pnc_run_v4<T, 2>(p, st) : a.taps == 3 ? pnc_run_v4<T, 3>(p, st) : pnc_run_v4<T, 4>(p, st);
    if (rc) return rc;
    if (a.S > 1 && a.taps > 1)
      TPX_CUDA_OK(launch_pdl(pnc_state_kernel, dim3((unsigned)((a.D + 255) / 256), (unsigned)a.B), dim3(256), 0, st, (const float*)a.x_out, a.state,
                             (int)a.S, (int)a.D, a.taps - 1));
    return TPX_OK;
  }
  if (a.S == 1) {
    TPX_CUDA_OK(launch_pdl(pnc_token_kernel<T>, dim3((unsigned)a.B), dim3(kPncThreads), 0, st, p));
    return TPX_OK;
  }
  const dim3 grid((unsigned)((a.S + kPncTokens - 1) / kPncTokens), (unsigned)a.B);
  TPX_CUDA_OK(launch_pdl(pnc_tokens_kernel<T>, grid, dim3(kPncThreads), 0, st, p));
  if (a.conv && a.taps > 1)
    TPX_CUDA_OK(launch_pdl(pnc_state_kernel, dim3((unsigned)((a.D + 255) / 256), (unsigned)a.B), dim3(256), 0, st, (const float*)a.x_out, a.state,
                           (int)a.S, (int)a.D, a.taps - 1));
  return TPX_OK;
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_postnorm_conv(const TpxPostnormConv* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "postnorm_conv: null argument block");
  TPX_REQUIRE(a->B >= 0 && a->S >= 0 && a->D > 0 && a->B <= 65535 && a->past >= 0, TPX_ERR_ARG, "postnorm_conv: bad shape");
  TPX_REQUIRE(a->S < (1 << 24) && a->D < (1 << 20) && a->past < (1ll << 30), TPX_ERR_ARG, "postnorm_conv: shape too large");
  if (a->B == 0 || a->S == 0) return TPX_OK;
  TPX_REQUIRE(a->x_out && (a->ids ? a->embed != nullptr : a->x && a->y && a->w), TPX_ERR_ARG, "postnorm_conv: null pointer");
  TPX_REQUIRE(!a->conv || (a->h && a->ldh >= a->D && a->taps >= 1 && a->taps <= kPncMaxTaps && (a->taps == 1 || a->state)), TPX_ERR_ARG,
              "postnorm_conv: the convolution needs h, 1 to %d taps and its state", kPncMaxTaps);
  TPX_REQUIRE(!a->dev_len || a->S == 1, TPX_ERR_ARG, "postnorm_conv: dev_len is for single tokens");
  return a->f32 ? pnc_run<float>(*a, (cudaStream_t)stream) : pnc_run<__nv_bfloat16>(*a, (cudaStream_t)stream);
}

extern "C" int tpx_postnorm_final(const TpxPostnormFinal* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "postnorm_final: null argument block");
  TPX_REQUIRE(a->n >= 0 && a->D > 0 && a->D < (1 << 20) && a->ldo >= a->D, TPX_ERR_ARG, "postnorm_final: bad shape");
  if (a->n == 0) return TPX_OK;
  TPX_REQUIRE(a->x && a->y && a->w && a->w_final && a->rows && a->out, TPX_ERR_ARG, "postnorm_final: null pointer");
  if (a->f32)
    TPX_CUDA_OK(launch_pdl(pnc_final_kernel<float>, dim3((unsigned)a->n), dim3(256), 0, (cudaStream_t)stream, a->x, a->y, a->w, a->w_final, a->rows,
                           (float*)a->out, (int)a->D, (int)a->ldo, a->alpha, a->eps));
  else
    TPX_CUDA_OK(launch_pdl(pnc_final_kernel<__nv_bfloat16>, dim3((unsigned)a->n), dim3(256), 0, (cudaStream_t)stream, a->x, a->y, a->w, a->w_final,
                           a->rows, (__nv_bfloat16*)a->out, (int)a->D, (int)a->ldo, a->alpha, a->eps));
  return TPX_OK;
}

extern "C" int tpx_argmax_f32(const float* x, int64_t rows, int64_t n, int64_t* out, void* stream) {
  TPX_REQUIRE(rows >= 0 && n > 0, TPX_ERR_ARG, "argmax_f32: bad shape");
  if (rows == 0) return TPX_OK;
  TPX_REQUIRE(x && out, TPX_ERR_ARG, "argmax_f32: null pointer");
  TPX_CUDA_OK(launch_pdl(argmax_f32_kernel, dim3((unsigned)rows), dim3(256), 0, (cudaStream_t)stream, x, (long long)n,
                         reinterpret_cast<long long*>(out)));
  return TPX_OK;
}
