// Latent attention (keys and values as two linear maps of one cached low-rank latent per token, plus a rotated key part
// shared by all heads) with a sliding window and a per-head output gate: preparation of queries and latents, the page cache,
// and attention in the latent space, where the key map is applied to the query and the value map to the weighted latents,
// so that a cached token is read once for all heads.
#include "tpx_hybrid.cuh"

namespace tpx {

// ---------------------------------------------------------------- norms, rotation, cache append: a CTA per token
constexpr int kPrepThreads = 256;
template <typename T>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(TpxLatentPrep p) {
  __shared__ float red[2][kPrepThreads / 32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int b = (int)(row / p.S), s = (int)(row % p.S);
  const int q_rank = (int)p.q_rank, kv_rank = (int)p.kv_rank, krp = (int)p.krp, rot = (int)p.rot_dim;
  const float* __restrict__ x = p.proj + row * p.ldp;
  const float* __restrict__ xk = x + q_rank;
  const int64_t past = p.dev_len ? *p.dev_len : p.past;
  const int64_t t = past + s;
  const int64_t pos = t - (p.start ? p.start[b] : 0);  // negative: padding
  // angles: the product position * frequency and its reduction to one turn in double, the functions in 32-bit
  float2* cs = reinterpret_cast<float2*>(p.cos_sin) + row * (rot / 2);
  for (int i = threadIdx.x; i < rot / 2; i += kPrepThreads) {
    const double turns = (double)(pos > 0 ? pos : 0) * p.freq[i] * 0.15915494309189533577;
    float sn, c;
    sincospif((float)(2.0 * (turns - rint(turns))), &sn, &c);
    cs[i] = make_float2(c, sn);
  }
  float sq = 0.0f, sk = 0.0f;
#pragma unroll 4
  for (int i = threadIdx.x; i < q_rank; i += kPrepThreads) sq = fmaf(x[i], x[i], sq);
  if (p.own_kv)
    for (int i = threadIdx.x; i < kv_rank; i += kPrepThreads) sk = fmaf(xk[i], xk[i], sk);
  sq = hy_warp_sum(sq);
  sk = hy_warp_sum(sk);
  if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sk; }
  __syncthreads();  // also publishes cs within the block
  sq = sk = 0.0f;
#pragma unroll
  for (int i = 0; i < kPrepThreads / 32; i++) { sq += red[0][i]; sk += red[1][i]; }
  const float qi = 1.0f / sqrtf(sq / (float)q_rank + p.eps);
  T* cq = reinterpret_cast<T*>(p.cq) + row * p.ldq;
#pragma unroll 4
  for (int i = threadIdx.x; i < p.ldq; i += kPrepThreads) hy_st(cq + i, i < q_rank ? x[i] * qi * p.q_norm[i] : 0.0f);
  if (p.own_kv) {
    const float ki = 1.0f / sqrtf(sk / (float)kv_rank + p.eps);
    T* lat = p.lat ? reinterpret_cast<T*>(p.lat) + ((int64_t)b * p.L + (p.L - p.S) + s) * p.R : nullptr;
    // of the call's tokens only the last npages blocks stay in the cache: the others would be overwritten
    const int64_t last_block = (past + p.S - 1) / 32;
    T* page = t / 32 > last_block - p.npages
                  ? reinterpret_cast<T*>(p.pages[(t / 32) % p.npages]) + ((int64_t)b * 32 + t % 32) * p.R : nullptr;
    for (int i = threadIdx.x; i < p.R; i += kPrepThreads) {
      float v = 0.0f;
      if (i < kv_rank) {
        v = xk[i] * ki * p.kv_norm[i];
      } else if (i >= krp && i < krp + rot) {
        const int e = i - krp;
        const float2 r = cs[e >> 1];
        const float u = xk[kv_rank + (e & ~1)], w = xk[kv_rank + (e | 1)];
        v = (e & 1) ? w * r.x + u * r.y : u * r.x - w * r.y;
      }
      if (pos < 0) v = 0.0f;
      if (lat) hy_st(lat + i, v);
      if (page) hy_st(page + i, v);
    }
    xk += kv_rank + rot;
  }
  for (int i = threadIdx.x; i < p.heads; i += kPrepThreads) p.gate[row * p.heads + i] = hy_sigmoid(xk[i]);
}

template <typename T>
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint64_t* pages, int64_t npages, int64_t R, int64_t past, int64_t n, int64_t L,
                                                            T* __restrict__ lat) {
  pdl_trigger();
  pdl_wait();
  const int64_t i = blockIdx.x, b = blockIdx.y, t = past - n + i;
  const T* src = reinterpret_cast<const T*>(pages[(t / 32) % npages]) + (b * 32 + t % 32) * R;
  T* dst = lat + (b * L + i) * R;
  for (int64_t e = threadIdx.x; e < R; e += 128) dst[e] = src[e];
}

// ---------------------------------------------------------------- the key map applied to the query
constexpr int kAbsTok = 8;
template <typename T>
__global__ void __launch_bounds__(128) latent_absorb_kernel(TpxLatentAbsorb p) {
  extern __shared__ float ab_q[];  // [kAbsTok][dim]
  pdl_trigger();
  pdl_wait();
  const int head = blockIdx.x;
  const int64_t t0 = (int64_t)blockIdx.z * kAbsTok;
  const int n = (int)min((int64_t)kAbsTok, p.T - t0);
  const int dim = (int)p.dim;
  const T* q = reinterpret_cast<const T*>(p.q) + t0 * p.ldq + (int64_t)head * (p.dim + p.rot_dim);
  for (int i = threadIdx.x; i < kAbsTok * dim; i += 128) {
    const int j = i / dim, d = i % dim;
    ab_q[i] = j < n ? hy_ld(q + j * p.ldq + d) : 0.0f;
  }
  __syncthreads();
  T* qa = reinterpret_cast<T*>(p.qa) + (t0 * p.heads + head) * p.R;
  const int64_t rs = p.heads * p.R;
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (c < p.krp) {
    float acc[kAbsTok] = {};
    if (c < p.kv_rank) {
      const T* w = reinterpret_cast<const T*>(p.w_uk) + (int64_t)head * dim * p.krp + c;
#pragma unroll 4
      for (int d = 0; d < dim; d++) {
        const float wv = hy_ld(w + (int64_t)d * p.krp);
#pragma unroll
        for (int j = 0; j < kAbsTok; j++) acc[j] = fmaf(ab_q[j * dim + d], wv, acc[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < kAbsTok; j++)
      if (j < n) hy_st(qa + j * rs + c, acc[j]);
  }
  if (blockIdx.y == 0) {
    const int rw = (int)(p.R - p.krp), half = (int)p.rot_dim / 2;
    for (int i = threadIdx.x; i < n * rw; i += 128) {
      const int j = i / rw, e = i % rw;
      float v = 0.0f;
      if (e < p.rot_dim) {
        const float2 r = reinterpret_cast<const float2*>(p.cos_sin)[(t0 + j) * half + (e >> 1)];
        const T* qr = q + j * p.ldq + dim;
        const float u = hy_ld(qr + (e & ~1)), w = hy_ld(qr + (e | 1));
        v = (e & 1) ? w * r.x + u * r.y : u * r.x - w * r.y;
      }
      hy_st(qa + j * rs + p.krp + e, v);
    }
  }
}

// ---------------------------------------------------------------- attention, any type and size: a warp per (token, head)
template <typename T, int NR>
__global__ void __launch_bounds__(128) latent_attn_kernel(TpxLatentAttn p) {
  pdl_trigger();
  pdl_wait();
  const int64_t item = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= p.B * p.S * p.heads) return;
  const int64_t row = item / p.heads;
  const int b = (int)(row / p.S), s = (int)(row % p.S);
  const int64_t past = p.dev_len ? *p.dev_len : p.past;
  const int64_t t = past + s, first = p.start ? p.start[b] : 0;
  const int64_t lo = max(first, t - p.window + 1);
  float q[NR], acc[NR];
  const T* qr = reinterpret_cast<const T*>(p.qa) + item * p.R;
#pragma unroll
  for (int i = 0; i < NR; i++) {
    const int e = i * 32 + lane;
    q[i] = e < p.R ? hy_ld(qr + e) * p.scale : 0.0f;
    acc[i] = 0.0f;
  }
  float m = -INFINITY, l = 0.0f;
  for (int64_t j = lo; j <= t; j++) {
    const T* kr = p.lat ? reinterpret_cast<const T*>(p.lat) + ((int64_t)b * p.L + (j - (past + p.S - p.L))) * p.R
                        : reinterpret_cast<const T*>(p.pages[(j / 32) % p.npages]) + ((int64_t)b * 32 + j % 32) * p.R;
    float k[NR], d = 0.0f;
#pragma unroll
    for (int i = 0; i < NR; i++) {
      const int e = i * 32 + lane;
      k[i] = e < p.R ? hy_ld(kr + e) : 0.0f;
      d = fmaf(q[i], k[i], d);
    }
    d = hy_warp_sum(d);
    const float mn = fmaxf(m, d), al = expf(m - mn), pr = expf(d - mn);
    l = fmaf(l, al, pr);
    m = mn;
#pragma unroll
    for (int i = 0; i < NR; i++) acc[i] = fmaf(acc[i], al, pr * k[i]);
  }
  const float inv = l > 0.0f ? 1.0f / l : 0.0f;
  T* o = reinterpret_cast<T*>(p.ol) + item * p.krp;
#pragma unroll
  for (int i = 0; i < NR; i++) {
    const int e = i * 32 + lane;
    if (e < p.krp) hy_st(o + e, acc[i] * inv);
  }
}

// ---------------------------------------------------------------- the value map and the output gate
template <typename T>
__global__ void __launch_bounds__(256) latent_value_kernel(TpxLatentValue p) {
  extern __shared__ float lv_o[];  // [kAbsTok][krp]
  pdl_trigger();
  pdl_wait();
  const int head = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t t0 = (int64_t)blockIdx.z * kAbsTok;
  const int n = (int)min((int64_t)kAbsTok, p.T - t0);
  const int krp = (int)p.krp;
  for (int i = threadIdx.x; i < kAbsTok * krp; i += 256) {
    const int j = i / krp;
    lv_o[i] = j < n ? hy_ld(reinterpret_cast<const T*>(p.ol) + ((t0 + j) * p.heads + head) * krp + i % krp) : 0.0f;
  }
  __syncthreads();
  T* out = reinterpret_cast<T*>(p.out);
  for (int e = blockIdx.y * 32 + warp; e < min((int)p.vdim, (int)blockIdx.y * 32 + 32); e += 8) {
    const T* w = reinterpret_cast<const T*>(p.w_uv) + ((int64_t)head * p.vdim + e) * krp;
    float acc[kAbsTok] = {};
    for (int c = lane; c < krp; c += 32) {
      const float wv = hy_ld(w + c);
#pragma unroll
      for (int j = 0; j < kAbsTok; j++) acc[j] = fmaf(lv_o[j * krp + c], wv, acc[j]);
    }
#pragma unroll
    for (int j = 0; j < kAbsTok; j++) {
      const float v = hy_warp_sum(acc[j]);
      if (lane == 0 && j < n) hy_st(out + (t0 + j) * p.ldo + (int64_t)head * p.vdim + e, v * p.gate[(t0 + j) * p.heads + head]);
    }
  }
  if (head == 0 && blockIdx.y == 0)
    for (int j = 0; j < n; j++)
      for (int64_t c = p.heads * p.vdim + threadIdx.x; c < p.ldo; c += 256) hy_st(out + (t0 + j) * p.ldo + c, 0.0f);
}

template <typename T>
static int latent_attn_plain(const TpxLatentAttn& a, cudaStream_t st) {
  const int64_t items = a.B * a.S * a.heads;
  const dim3 grid((unsigned)((items + 3) / 4));
  void (*k)(TpxLatentAttn) = latent_attn_kernel<T, 36>;
  if (a.R <= 128) k = latent_attn_kernel<T, 4>;
  else if (a.R <= 256) k = latent_attn_kernel<T, 8>;
  else if (a.R <= 640) k = latent_attn_kernel<T, 20>;
  TPX_CUDA_OK(launch_pdl(k, grid, dim3(128), 0, st, a));
  return TPX_OK;
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_latent_prep(const TpxLatentPrep* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "latent_prep: null argument block");
  TPX_REQUIRE(a->B >= 0 && a->S >= 0 && a->q_rank > 0 && a->kv_rank > 0 && a->rot_dim >= 0 && a->rot_dim % 2 == 0 && a->heads > 0 && a->past >= 0,
              TPX_ERR_ARG, "latent_prep: bad shape");
  if (a->B * a->S == 0) return TPX_OK;
  TPX_REQUIRE(a->proj && a->q_norm && a->cq && a->gate && (a->rot_dim == 0 || (a->freq && a->cos_sin)), TPX_ERR_ARG, "latent_prep: null pointer");
  TPX_REQUIRE(!a->own_kv || (a->kv_norm && a->pages && a->npages > 0), TPX_ERR_ARG, "latent_prep: a layer with its own latent needs its cache");
  TPX_REQUIRE(a->krp >= a->kv_rank && a->R >= a->krp + a->rot_dim && a->ldq >= a->q_rank && a->L >= (a->lat ? a->S : 0), TPX_ERR_ARG,
              "latent_prep: a row is smaller than its contents");
  TPX_REQUIRE(!a->dev_len || a->S == 1, TPX_ERR_ARG, "latent_prep: dev_len is for single tokens");
  const dim3 grid((unsigned)(a->B * a->S));
  if (a->f32) TPX_CUDA_OK(launch_pdl(latent_prep_kernel<float>, grid, dim3(kPrepThreads), 0, (cudaStream_t)stream, *a));
  else TPX_CUDA_OK(launch_pdl(latent_prep_kernel<__nv_bfloat16>, grid, dim3(kPrepThreads), 0, (cudaStream_t)stream, *a));
  return TPX_OK;
}

extern "C" int tpx_latent_gather(const uint64_t* pages, int64_t npages, int64_t B, int64_t R, int64_t past, int64_t n, int64_t L, void* lat, int f32,
                                 void* stream) {
  TPX_REQUIRE(npages > 0 && B >= 0 && R > 0 && n >= 0 && past >= n && L >= n && B <= 65535, TPX_ERR_ARG, "latent_gather: bad shape");
  if (B == 0 || n == 0) return TPX_OK;
  TPX_REQUIRE(pages && lat, TPX_ERR_ARG, "latent_gather: null pointer");
  const dim3 grid((unsigned)n, (unsigned)B);
  if (f32) TPX_CUDA_OK(launch_pdl(latent_gather_kernel<float>, grid, dim3(128), 0, (cudaStream_t)stream, pages, npages, R, past, n, L, (float*)lat));
  else TPX_CUDA_OK(launch_pdl(latent_gather_kernel<uint16_t>, grid, dim3(128), 0, (cudaStream_t)stream, pages, npages, R, past, n, L, (uint16_t*)lat));
  return TPX_OK;
}

extern "C" int tpx_latent_absorb(const TpxLatentAbsorb* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "latent_absorb: null argument block");
  TPX_REQUIRE(a->T >= 0 && a->heads > 0 && a->dim > 0 && a->kv_rank > 0 && a->krp >= a->kv_rank && a->R >= a->krp + a->rot_dim &&
                  a->ldq >= a->heads * (a->dim + a->rot_dim), TPX_ERR_ARG, "latent_absorb: bad shape");
  TPX_REQUIRE(a->dim <= 1024, TPX_ERR_UNSUPPORTED, "latent_absorb: heads of at most 1024 channels");
  if (a->T == 0) return TPX_OK;
  TPX_REQUIRE(a->q && a->w_uk && a->qa && (a->rot_dim == 0 || a->cos_sin), TPX_ERR_ARG, "latent_absorb: null pointer");
  if (latent_absorb_mma_serves(*a)) return latent_absorb_mma(*a, (cudaStream_t)stream);
  const int64_t tz = (a->T + kAbsTok - 1) / kAbsTok;
  TPX_REQUIRE(tz <= 65535, TPX_ERR_UNSUPPORTED, "latent_absorb: too many tokens in one call");
  const dim3 grid((unsigned)a->heads, (unsigned)((a->krp + 127) / 128), (unsigned)tz);
  const size_t smem = (size_t)kAbsTok * a->dim * 4;
  if (a->f32) TPX_CUDA_OK(launch_pdl(latent_absorb_kernel<float>, grid, dim3(128), smem, (cudaStream_t)stream, *a));
  else TPX_CUDA_OK(launch_pdl(latent_absorb_kernel<__nv_bfloat16>, grid, dim3(128), smem, (cudaStream_t)stream, *a));
  return TPX_OK;
}

extern "C" int tpx_latent_attn(const TpxLatentAttn* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "latent_attn: null argument block");
  TPX_REQUIRE(a->B >= 0 && a->S >= 0 && a->heads > 0 && a->krp > 0 && a->R >= a->krp && a->window > 0 && a->past >= 0, TPX_ERR_ARG,
              "latent_attn: bad shape");
  TPX_REQUIRE(a->R <= 1152, TPX_ERR_UNSUPPORTED, "latent_attn: rows of at most 1152 elements, got %ld", (long)a->R);
  if (a->B * a->S == 0) return TPX_OK;
  TPX_REQUIRE(a->qa && a->ol, TPX_ERR_ARG, "latent_attn: null pointer");
  TPX_REQUIRE(a->lat ? a->L >= a->S + (a->window - 1 < a->past ? a->window - 1 : a->past)
                     : a->S == 1 && a->pages && a->npages > 0, TPX_ERR_ARG, "latent_attn: the keys of the window are not there");
  TPX_REQUIRE(!a->dev_len || a->S == 1, TPX_ERR_ARG, "latent_attn: dev_len is for single tokens");
  if (latent_decode_serves(*a)) return latent_decode(*a, (cudaStream_t)stream);
  return a->f32 ? latent_attn_plain<float>(*a, (cudaStream_t)stream) : latent_attn_plain<__nv_bfloat16>(*a, (cudaStream_t)stream);
}

extern "C" int tpx_latent_value(const TpxLatentValue* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "latent_value: null argument block");
  TPX_REQUIRE(a->T >= 0 && a->heads > 0 && a->vdim > 0 && a->krp > 0 && a->krp <= 1152 && a->ldo >= a->heads * a->vdim, TPX_ERR_ARG, "latent_value: bad shape");
  if (a->T == 0) return TPX_OK;
  TPX_REQUIRE(a->ol && a->gate && a->w_uv && a->out, TPX_ERR_ARG, "latent_value: null pointer");
  if (latent_value_mma_serves(*a)) return latent_value_mma(*a, (cudaStream_t)stream);
  const int64_t tz = (a->T + kAbsTok - 1) / kAbsTok;
  TPX_REQUIRE(tz <= 65535, TPX_ERR_UNSUPPORTED, "latent_value: too many tokens in one call");
  const dim3 grid((unsigned)a->heads, (unsigned)((a->vdim + 31) / 32), (unsigned)tz);
  const size_t smem = (size_t)kAbsTok * a->krp * 4;
  if (a->f32) TPX_CUDA_OK(launch_pdl(latent_value_kernel<float>, grid, dim3(256), smem, (cudaStream_t)stream, *a));
  else TPX_CUDA_OK(launch_pdl(latent_value_kernel<__nv_bfloat16>, grid, dim3(256), smem, (cudaStream_t)stream, *a));
  return TPX_OK;
}
