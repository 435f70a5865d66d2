// Chunked differential attention with capped scores: the page cache, the kernel for any type and size, and the entry point.
// Two softmax attentions ("maps") with queries and keys of their own share the values; a head's output is map 1 minus lambda
// times map 2, over its root mean square. A token sees its own chunk of the sequence only, so that a layer's page table stops
// growing at the pages a chunk can touch.
#include "tpx_hybrid.cuh"

namespace tpx {

// ---------------------------------------------------------------- cache: a CTA per (token, key / value head)
template <typename T>
__global__ void __launch_bounds__(128) diff_append_kernel(TpxDiffAttn p) {
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x, g = blockIdx.y, b = row / p.S, s = row % p.S;
  const int64_t past = p.dev_len ? *p.dev_len : p.past, t = past + s;
  const int dim = (int)p.dim, dp = (dim + 15) / 16 * 16, vdim = (int)p.vdim;
  const T* pr = reinterpret_cast<const T*>(p.proj) + row * p.ldp;
  // of the call's tokens only the last npages blocks stay in the cache: the others would be overwritten
  const bool keep = t / 32 > (past + p.S - 1) / 32 - p.npages;
  T* page = keep ? reinterpret_cast<T*>(p.pages[(t / 32) % p.npages]) + ((b * p.kv_heads + g) * 32 + t % 32) * p.R : nullptr;
  T* live = p.live ? reinterpret_cast<T*>(p.live) + ((b * p.L + (p.L - p.S) + s) * p.kv_heads + g) * p.R : nullptr;
  if (!page && !live) return;
  for (int i = threadIdx.x; i < p.R; i += 128) {
    float v = 0.0f;
    const int m = i / dp, c = i % dp;
    if (m < 2) {
      if (c < dim) v = hy_ld(pr + p.k_col + (g * 2 + m) * dim + c);
    } else if (i - 2 * dp < vdim) {
      v = hy_ld(pr + p.v_col + g * vdim + (i - 2 * dp));
    }
    if (page) hy_st(page + i, v);
    if (live) hy_st(live + i, v);
  }
}

// The same in 16-byte units, for bf16 head sizes that are multiples of 8: a thread per unit of a row.
__global__ void __launch_bounds__(256) diff_append_v8_kernel(TpxDiffAttn p, int64_t row0) {
  pdl_trigger();
  pdl_wait();
  const int ur = (int)p.R / 8, d8 = (int)p.dim / 8, dp8 = (int)((p.dim + 15) / 16 * 2), v8 = (int)p.vdim / 8, G = (int)p.kv_heads;
  const int64_t idx = (int64_t)blockIdx.x * 256 + threadIdx.x;
  const int64_t rg = idx / ur;  // (sequence, token from row0 on, head)
  const int u = (int)(idx % ur), g = (int)(rg % G);
  const int64_t n = p.S - row0, bs = rg / G, b = bs / n, s = row0 + bs % n;
  if (b >= p.B) return;
  const int64_t past = p.dev_len ? *p.dev_len : p.past, t = past + s;
  const uint4* pr = reinterpret_cast<const uint4*>(reinterpret_cast<const uint16_t*>(p.proj) + (b * p.S + s) * p.ldp);
  const int m = u / dp8, c = u % dp8;
  uint4 v = make_uint4(0, 0, 0, 0);
  if (m < 2) {
    if (c < d8) v = pr[p.k_col / 8 + (g * 2 + m) * d8 + c];
  } else if (u - 2 * dp8 < v8) {
    v = pr[p.v_col / 8 + g * v8 + u - 2 * dp8];
  }
  if (t / 32 > (past + p.S - 1) / 32 - p.npages)
    reinterpret_cast<uint4*>(p.pages[(t / 32) % p.npages])[((b * G + g) * 32 + t % 32) * ur + u] = v;
  if (p.live) reinterpret_cast<uint4*>(p.live)[((b * p.L + (p.L - p.S) + s) * G + g) * ur + u] = v;
}

// the cached tokens past - n .. past - 1 into rows 0 .. n - 1 of live; runs before the append, which may use their pages again
template <typename T>
__global__ void __launch_bounds__(128) diff_gather_kernel(TpxDiffAttn p) {
  pdl_trigger();
  pdl_wait();
  const int64_t i = blockIdx.x, g = blockIdx.y, b = blockIdx.z, t = p.past - (p.L - p.S) + i;
  const T* src = reinterpret_cast<const T*>(p.pages[(t / 32) % p.npages]) + ((b * p.kv_heads + g) * 32 + t % 32) * p.R;
  T* dst = reinterpret_cast<T*>(p.live) + ((b * p.L + i) * p.kv_heads + g) * p.R;
  for (int e = threadIdx.x; e < p.R; e += 128) dst[e] = src[e];
}

// ---------------------------------------------------------------- attention, any type and size: a warp per (token, head)
// Lanes hold a key each for the scores and NR value columns each for the sums.
constexpr int kDiffWarps = 4;

template <typename T, int NR>
__global__ void __launch_bounds__(kDiffWarps * 32) diff_attn_kernel(TpxDiffAttn p) {
  extern __shared__ float df_q[];  // [warps][2 dim]
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t item = (int64_t)blockIdx.x * kDiffWarps + warp;
  const int64_t row = item / p.heads;
  const int head = (int)(item % p.heads), dim = (int)p.dim, vdim = (int)p.vdim, dp = (dim + 15) / 16 * 16;
  if (row >= p.B * p.S) return;
  const int64_t b = row / p.S, g = head / (p.heads / p.kv_heads);
  const int64_t past = p.dev_len ? *p.dev_len : p.past, t = past + row % p.S;
  const int64_t start = p.start ? p.start[b] : 0;
  const int64_t lo = t < start ? t + 1 : start + (t - start) / p.chunk * p.chunk;  // padding sees nothing
  float* q = df_q + warp * 2 * dim;
  const T* pq = reinterpret_cast<const T*>(p.proj) + row * p.ldp + p.q_col + (int64_t)head * 2 * dim;
  for (int i = lane; i < 2 * dim; i += 32) q[i] = hy_ld(pq + i) * p.scale;
  __syncwarp();
  auto key = [&](int64_t j) -> const T* {
    if (p.live) return reinterpret_cast<const T*>(p.live) + ((b * p.L + j - (past - (p.L - p.S))) * p.kv_heads + g) * p.R;
    return reinterpret_cast<const T*>(p.pages[(j / 32) % p.npages]) + ((b * p.kv_heads + g) * 32 + j % 32) * p.R;
  };
  float o[2][NR] = {}, mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
  for (int64_t j0 = lo; j0 <= t; j0 += 32) {
    const int n = (int)min((int64_t)32, t - j0 + 1);
    float s[2] = {-INFINITY, -INFINITY};
    if (lane < n) {
      const T* k = key(j0 + lane);
#pragma unroll
      for (int m = 0; m < 2; m++) {
        float a = 0.0f;
        for (int c = 0; c < dim; c++) a = fmaf(q[m * dim + c], hy_ld(k + m * dp + c), a);
        s[m] = p.softcap * tanhf(a / p.softcap);
      }
    }
    float e[2];
#pragma unroll
    for (int m = 0; m < 2; m++) {
      float x = s[m];
#pragma unroll
      for (int d = 16; d > 0; d >>= 1) x = fmaxf(x, __shfl_xor_sync(0xffffffffu, x, d));
      const float mn = fmaxf(mx[m], x), al = expf(mx[m] - mn);
      e[m] = lane < n ? expf(s[m] - mn) : 0.0f;
      sum[m] = sum[m] * al + hy_warp_sum(e[m]);
      mx[m] = mn;
#pragma unroll
      for (int i = 0; i < NR; i++) o[m][i] *= al;
    }
    for (int j = 0; j < n; j++) {
      const T* v = key(j0 + j) + 2 * dp;
      const float e1 = __shfl_sync(0xffffffffu, e[0], j), e2 = __shfl_sync(0xffffffffu, e[1], j);
#pragma unroll
      for (int i = 0; i < NR; i++)
        if (lane + 32 * i < vdim) {
          const float x = hy_ld(v + lane + 32 * i);
          o[0][i] = fmaf(e1, x, o[0][i]);
          o[1][i] = fmaf(e2, x, o[1][i]);
        }
    }
  }
  const float i1 = sum[0] > 0.0f ? 1.0f / sum[0] : 0.0f, i2 = sum[1] > 0.0f ? 1.0f / sum[1] : 0.0f;
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NR; i++) {
    o[0][i] = o[0][i] * i1 - p.lambda * (o[1][i] * i2);
    ss = fmaf(o[0][i], o[0][i], ss);
  }
  const float inv = p.mult / sqrtf(hy_warp_sum(ss) / (float)vdim + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + row * p.ldo + (int64_t)head * vdim;
#pragma unroll
  for (int i = 0; i < NR; i++)
    if (lane + 32 * i < vdim) hy_st(out + lane + 32 * i, o[0][i] * inv);
}

template <typename T>
static int diff_run(const TpxDiffAttn& a, cudaStream_t st) {
  const int64_t nr = (a.vdim + 31) / 32;
  void (*k)(TpxDiffAttn) = nr <= 1 ? diff_attn_kernel<T, 1> : nr <= 2 ? diff_attn_kernel<T, 2> : nr <= 4 ? diff_attn_kernel<T, 4>
                           : nr <= 8 ? diff_attn_kernel<T, 8> : diff_attn_kernel<T, 16>;
  const int64_t items = a.B * a.S * a.heads;
  TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)((items + kDiffWarps - 1) / kDiffWarps)), dim3(kDiffWarps * 32), (size_t)kDiffWarps * 2 * a.dim * 4, st, a));
  return TPX_OK;
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_diff_prefill_serves(int64_t dim, int64_t vdim, float softcap) { return diff_prefill_serves(dim, vdim, softcap); }

extern "C" int tpx_diff_attn(const TpxDiffAttn* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "diff_attn: null argument block");
  TPX_REQUIRE(a->B >= 0 && a->S >= 0 && a->L >= a->S && a->heads > 0 && a->kv_heads > 0 && a->heads % a->kv_heads == 0 && a->dim > 0 && a->vdim > 0 &&
                  a->chunk > 0 && a->npages > 0 && a->past >= a->L - a->S && a->softcap > 0.0f, TPX_ERR_ARG, "diff_attn: bad shape");
  TPX_REQUIRE(a->dim <= 512 && a->vdim <= 512, TPX_ERR_UNSUPPORTED, "diff_attn: heads of at most 512 channels, got %ld, %ld", (long)a->dim, (long)a->vdim);
  TPX_REQUIRE(a->B <= 65535 && a->S < (1 << 24) && a->past < (1ll << 30) && a->chunk < (1ll << 30) && a->heads < (1 << 15) && a->B * a->S * a->heads < (1ll << 31),
              TPX_ERR_ARG, "diff_attn: shape too large");
  if (a->B == 0 || a->S == 0) return TPX_OK;
  TPX_REQUIRE(a->proj && a->pages && a->out, TPX_ERR_ARG, "diff_attn: null pointer");
  const int64_t dp = (a->dim + 15) / 16 * 16;
  TPX_REQUIRE(a->R == 2 * dp + (a->vdim + 15) / 16 * 16 + 8, TPX_ERR_ARG, "diff_attn: cache rows of %ld elements do not fit the head sizes", (long)a->R);
  TPX_REQUIRE(a->q_col >= 0 && a->k_col >= 0 && a->v_col >= 0 && a->q_col + a->heads * 2 * a->dim <= a->ldp && a->k_col + a->kv_heads * 2 * a->dim <= a->ldp &&
                  a->v_col + a->kv_heads * a->vdim <= a->ldp && a->ldo >= a->heads * a->vdim, TPX_ERR_ARG, "diff_attn: columns outside their rows");
  TPX_REQUIRE(!a->dev_len || a->S == 1, TPX_ERR_ARG, "diff_attn: dev_len is for single tokens");
  const int64_t reach = a->chunk - 1 < a->past ? a->chunk - 1 : a->past;
  // pages: all tokens in reach of the last one, or of the one after it
  TPX_REQUIRE(a->dev_len || a->npages * 32 >= (a->past + a->S < a->chunk ? a->past + a->S : a->chunk), TPX_ERR_ARG, "diff_attn: the page table is too short");
  cudaStream_t st = (cudaStream_t)stream;
  if (a->S == 1) {
    if (diff_decode_serves(*a)) return diff_decode(*a, st);
  } else {
    TPX_REQUIRE(a->L - a->S >= reach, TPX_ERR_ARG, "diff_attn: the keys in reach are not there");
    TPX_REQUIRE(a->live || (a->L == a->S && !a->f32 && diff_prefill_serves(a->dim, a->vdim, a->softcap)), TPX_ERR_ARG, "diff_attn: working space is missing");
    if (a->L > a->S) {
      void (*k)(TpxDiffAttn) = a->f32 ? diff_gather_kernel<float> : diff_gather_kernel<__nv_bfloat16>;
      TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)(a->L - a->S), (unsigned)a->kv_heads, (unsigned)a->B), dim3(128), 0, st, *a));
    }
  }
  if (!a->f32 && a->dim % 8 == 0 && a->vdim % 8 == 0 && a->ldp % 8 == 0 && a->k_col % 8 == 0 && a->v_col % 8 == 0 && (((uintptr_t)a->proj | (uintptr_t)a->live) & 15) == 0) {
    // tokens whose pages the call's later tokens use again need no rows, unless they go to `live`
    int64_t row0 = a->live || a->dev_len ? 0 : (((a->past + a->S - 1) / 32 - a->npages + 1) * 32 - a->past);
    if (row0 < 0) row0 = 0;
    const int64_t units = a->B * (a->S - row0) * a->kv_heads * (a->R / 8);
    TPX_REQUIRE(units < (1ll << 38), TPX_ERR_ARG, "diff_attn: shape too large");
    TPX_CUDA_OK(launch_pdl(diff_append_v8_kernel, dim3((unsigned)((units + 255) / 256)), dim3(256), 0, st, *a, row0));
  } else {
    TPX_REQUIRE(a->kv_heads <= 65535, TPX_ERR_UNSUPPORTED, "diff_attn: too many heads");
    void (*k)(TpxDiffAttn) = a->f32 ? diff_append_kernel<float> : diff_append_kernel<__nv_bfloat16>;
    TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)(a->B * a->S), (unsigned)a->kv_heads), dim3(128), 0, st, *a));
  }
  if (a->S > 1 && !a->f32 && diff_prefill_serves(a->dim, a->vdim, a->softcap)) return diff_prefill(*a, st);
  TpxDiffAttn b = *a;
  if (a->S == 1) b.live = nullptr;
  return a->f32 ? diff_run<float>(b, st) : diff_run<__nv_bfloat16>(b, st);
}
