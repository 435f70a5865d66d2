// Linear in true 32-bit: fp32 operands, fp32 products and sums on the CUDA cores (no reduced-precision tensor-core mode),
// for models that are run in float32; and the tpx_linear entry point that chooses between it and the tcgen05 kernel.
//
// 64 x 64 output tiles, 16 k values per step in shared memory, 4 x 4 outputs per thread. A decode step (few rows) takes
// one warp per output feature instead: a 64-row tile would be mostly empty.
#include "tpx_hybrid.cuh"

namespace tpx {

constexpr int kF32Tile = 64, kF32K = 16;

struct F32Epi {
  const float* bias;
  void* y;
  long long ldy;
  int out_f32, act, act_from;
  const float* ap;
  float* z;  // gated units
  const float *res, *add, *nw, *nb;
  float *x_out, *h;
  long long ldz, ldr, ldh;
  float limit, nalpha;
};
__device__ __forceinline__ bool f32_pairs(const F32Epi& e, int n) { return e.act == TPX_ACT_CLAMPED_GLU && n >= e.act_from; }

__device__ __forceinline__ void f32_finish(const F32Epi& e, long long m, int n, float v) {
  if (e.bias) v += e.bias[n];
  if (e.x_out) {
    v += e.res[m * e.ldr + n];
    if (e.add) v += e.add[n];
    e.x_out[m * e.ldr + n] = v;
    e.h[m * e.ldh + n] = fmaf(tanhf(e.nalpha * v), e.nw[n], e.nb[n]);
    return;
  }
  if (e.act && n >= e.act_from) v = hy_act(v, e.act, e.ap ? e.ap[0] : 0.0f, e.ap ? e.ap[1] : 0.0f);
  if (e.out_f32) reinterpret_cast<float*>(e.y)[m * e.ldy + n] = v;
  else reinterpret_cast<__nv_bfloat16*>(e.y)[m * e.ldy + n] = __float2bfloat16_rn(v);
}

// columns n (even distance from act_from) and n + 1: one gated unit
__device__ __forceinline__ void f32_finish_pair(const F32Epi& e, long long m, int n, float g, float u) {
  if (e.bias) { g += e.bias[n]; u += e.bias[n + 1]; }
  e.z[m * e.ldz + (n - e.act_from) / 2] = hy_clamped_glu(g, u, e.limit);
}

__global__ void __launch_bounds__(256) linear_f32_kernel(const float* __restrict__ w, const float* __restrict__ x, long long M, int N, int K,
                                                         long long ldw, long long ldx, F32Epi e) {
  __shared__ float xs[kF32K][kF32Tile + 4], ws[kF32K][kF32Tile + 4];
  pdl_trigger();
  pdl_wait();
  const long long m0 = (long long)blockIdx.y * kF32Tile;
  const int n0 = blockIdx.x * kF32Tile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kF32K) {
    for (int i = threadIdx.x; i < kF32Tile * kF32K; i += 256) {
      const int r = i / kF32K, c = i % kF32K;
      xs[c][r] = (m0 + r < M && k0 + c < K) ? x[(m0 + r) * ldx + k0 + c] : 0.0f;
      ws[c][r] = (n0 + r < N && k0 + c < K) ? w[(long long)(n0 + r) * ldw + k0 + c] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < kF32K; c++) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; i++) { a[i] = xs[c][ty * 4 + i]; b[i] = ws[c][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const long long m = m0 + ty * 4 + i;
      const int n = n0 + tx * 4 + j;
      if (m < M && n < N) {
        if (!f32_pairs(e, n)) f32_finish(e, m, n, acc[i][j]);
        else if (!(j & 1)) f32_finish_pair(e, m, n, acc[i][j], acc[i][j + 1]);
      }
    }
}

constexpr int kF32Rows = 4;
__global__ void __launch_bounds__(256) linear_f32_rows_kernel(const float* __restrict__ w, const float* __restrict__ x, long long M, int N, int K,
                                                              long long ldw, long long ldx, F32Epi e) {
  pdl_trigger();
  pdl_wait();
  const int n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const long long m0 = (long long)blockIdx.y * kF32Rows;
  if (n >= N) return;
  const bool pair = f32_pairs(e, n);
  if (pair && (n & 1)) return;  // with its neighbour
  float acc[kF32Rows] = {}, up[kF32Rows] = {};
  for (int k = lane; k < K; k += 32) {
    const float b = w[(long long)n * ldw + k], c = pair ? w[(long long)(n + 1) * ldw + k] : 0.0f;
#pragma unroll
    for (int i = 0; i < kF32Rows; i++)
      if (m0 + i < M) {
        const float v = x[(m0 + i) * ldx + k];
        acc[i] = fmaf(v, b, acc[i]);
        up[i] = fmaf(v, c, up[i]);
      }
  }
#pragma unroll
  for (int i = 0; i < kF32Rows; i++) {
    const float s = hy_warp_sum(acc[i]);
    if (pair) {
      const float u = hy_warp_sum(up[i]);
      if (lane == 0 && m0 + i < M) f32_finish_pair(e, m0 + i, n, s, u);
    } else if (lane == 0 && m0 + i < M) f32_finish(e, m0 + i, n, s);
  }
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_linear(const TpxLinear* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "linear: null argument block");
  TPX_REQUIRE(a->M >= 0 && a->N > 0 && a->K > 0, TPX_ERR_ARG, "linear: bad shape M=%ld N=%ld K=%ld", (long)a->M, (long)a->N, (long)a->K);
  if (a->M == 0) return TPX_OK;
  const bool glu = a->act == TPX_ACT_CLAMPED_GLU;
  const int64_t ny = glu ? a->act_from : a->N;  // columns of y
  TPX_REQUIRE(a->w && a->x && (a->y || a->x_out || ny == 0), TPX_ERR_ARG, "linear: null pointer");
  TPX_REQUIRE(a->ldw >= a->K && a->ldx >= a->K && (a->x_out || a->ldy >= ny), TPX_ERR_ARG, "linear: a leading dimension is smaller than its row");
  TPX_REQUIRE(a->M < (1 << 24) && a->N < (1 << 24) && a->K < (1 << 24), TPX_ERR_ARG, "linear: shape too large");
  TPX_REQUIRE(a->act >= TPX_ACT_NONE && a->act <= TPX_ACT_CLAMPED_GLU, TPX_ERR_ARG, "linear: unknown activation %d", a->act);
  TPX_REQUIRE(a->act != TPX_ACT_XIELU || a->act_params, TPX_ERR_ARG, "linear: xIELU needs its two parameters");
  TPX_REQUIRE(!glu || (a->z && !a->x_out && a->act_from % 2 == 0 && a->N % 2 == 0 && a->act_from >= 0 && a->act_from <= a->N &&
                       a->ldz >= (a->N - a->act_from) / 2), TPX_ERR_ARG, "linear: gated units need z and whole pairs of columns");
  TPX_REQUIRE(!a->x_out || (a->res && a->norm_w && a->norm_b && a->h && a->ldr >= a->N && a->ldh >= a->N && a->act == TPX_ACT_NONE), TPX_ERR_ARG,
              "linear: the residual form needs the stream, the norm and no activation");
  cudaStream_t st = (cudaStream_t)stream;
  if (!a->f32) return linear_tc_ex(*a, st);
  const F32Epi e = {a->bias, a->y, (long long)a->ldy, a->out_f32, a->act, a->act_from, a->act_params, (float*)a->z, a->res, a->add,
                    a->norm_w, a->norm_b, a->x_out, (float*)a->h, (long long)a->ldz, (long long)a->ldr, (long long)a->ldh, a->limit, a->norm_alpha};
  const float* w = (const float*)a->w;
  const float* x = (const float*)a->x;
  if (a->M <= 16) {
    TPX_CUDA_OK(launch_pdl(linear_f32_rows_kernel, dim3((unsigned)((a->N + 7) / 8), (unsigned)((a->M + kF32Rows - 1) / kF32Rows)), dim3(256), 0, st,
                           w, x, (long long)a->M, (int)a->N, (int)a->K, (long long)a->ldw, (long long)a->ldx, e));
  } else {
    const int64_t my = (a->M + kF32Tile - 1) / kF32Tile;
    TPX_REQUIRE(my <= 65535, TPX_ERR_UNSUPPORTED, "linear: too many rows for one 32-bit call");
    TPX_CUDA_OK(launch_pdl(linear_f32_kernel, dim3((unsigned)((a->N + kF32Tile - 1) / kF32Tile), (unsigned)my), dim3(256), 0, st, w, x,
                           (long long)a->M, (int)a->N, (int)a->K, (long long)a->ldw, (long long)a->ldx, e));
  }
  return TPX_OK;
}
