// Generalized delta rule (a linear recurrence with a matrix state per head), token by token in 32-bit:
//   S_t = diag(w_t) S_(t-1) - (a_t u_t)(u_t^T S_(t-1)) + k_t v_t^T,   o_t = S_t^T r_t,   u = k / sqrt(sum k^2 + 1e-6)
// A column of S (one value channel) evolves without the others: only the scalars u^T s and r^T s of the column are sums
// over key channels. So a CTA owns some columns of one (sequence, head); LPC = DP / 16 neighbouring lanes hold a column,
// 16 key channels each, in registers for the whole call. The vectors of 16 tokens at a time (decays, rates, unit keys: the
// exponentials and square roots) are prepared by all warps into shared memory.
// The read-outs go to `raw` in fp32; a second kernel divides each head by its root mean square and applies weight and gate.
#include "tpx_hybrid.cuh"

namespace tpx {

constexpr int kDeltaTok = 16;

template <typename T>
struct DeltaParams {
  const T* proj;
  const float *wraw, *a_bias;
  const int *start, *dev_len;
  float *state, *raw;
  int B, S, past, H, dim;
  long long ldp;
};

template <int DP>
struct DeltaCfg {
  static constexpr int LPC = DP / 16;                        // lanes per column
  static constexpr int COLS = (128 / LPC) < DP ? (128 / LPC) : DP;  // columns per CTA
  static constexpr int THREADS = COLS * LPC;
  static constexpr size_t SMEM = (size_t)kDeltaTok * (5 * DP + COLS) * 4;
};

template <typename T, int DP>
__global__ void __launch_bounds__(DeltaCfg<DP>::THREADS) delta_kernel(DeltaParams<T> p) {
  using C = DeltaCfg<DP>;
  extern __shared__ __align__(16) float dl_smem[];
  float* s_w = dl_smem;                      // decay           [tok][DP]
  float* s_u = s_w + kDeltaTok * DP;         // unit key
  float* s_a = s_u + kDeltaTok * DP;         // - rate * unit key
  float* s_k = s_a + kDeltaTok * DP;         // key
  float* s_r = s_k + kDeltaTok * DP;         // query
  float* s_v = s_r + kDeltaTok * DP;         // value           [tok][COLS]
  pdl_trigger();
  pdl_wait();
  const int head = blockIdx.x, c0 = blockIdx.y * C::COLS, b = blockIdx.z;
  const int l = threadIdx.x % C::LPC, cl = threadIdx.x / C::LPC, col = c0 + cl;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int NW = C::THREADS / 32 > 0 ? C::THREADS / 32 : 1;
  const int hd = p.H * p.dim;
  float* st = p.state + ((int64_t)(b * p.H + head) * p.dim) * p.dim + col;
  float s[16];
#pragma unroll
  for (int i = 0; i < 16; i++) {
    const int k = (i >> 2) * 4 * C::LPC + l * 4 + (i & 3);
    s[i] = (col < p.dim && k < p.dim) ? st[(int64_t)k * p.dim] : 0.0f;
  }
  const int past = p.dev_len ? *p.dev_len : p.past;
  const int first = p.start ? max(0, min(p.S, p.start[b] - past)) : 0;  // padding leaves the state alone
  for (int t0 = first; t0 < p.S; t0 += kDeltaTok) {
    const int n = min(kDeltaTok, p.S - t0);
    __syncthreads();
    for (int j = warp; j < n; j += NW) {
      const int64_t row = (int64_t)b * p.S + t0 + j;
      const T* pr = p.proj + row * p.ldp + head * p.dim;
      float ss = 0.0f;
      for (int i = lane; i < DP; i += 32) {
        const float k = i < p.dim ? hy_ld(pr + hd + i) : 0.0f;
        s_k[j * DP + i] = k;
        ss = fmaf(k, k, ss);
      }
      const float inv = 1.0f / sqrtf(hy_warp_sum(ss) + 1e-6f);
      for (int i = lane; i < DP; i += 32) {
        const bool in = i < p.dim;
        const float u = in ? hy_ld(pr + hd + i) * inv : 0.0f;
        const float rate = in ? hy_sigmoid(hy_ld(pr + 3 * hd + i) + p.a_bias[head * p.dim + i]) : 0.0f;
        s_u[j * DP + i] = u;
        s_a[j * DP + i] = -rate * u;
        s_r[j * DP + i] = in ? hy_ld(pr + i) : 0.0f;
        s_w[j * DP + i] = in ? expf(-0.60653065971263342f * hy_sigmoid(p.wraw[row * hd + head * p.dim + i])) : 0.0f;
      }
      for (int i = lane; i < C::COLS; i += 32) s_v[j * C::COLS + i] = c0 + i < p.dim ? hy_ld(pr + 2 * hd + c0 + i) : 0.0f;
    }
    __syncthreads();
    for (int j = 0; j < n; j++) {
      const float v = s_v[j * C::COLS + cl];
      float q4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      const float4* pu = reinterpret_cast<const float4*>(s_u + j * DP) + l;
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const float4 u = pu[i * C::LPC];
        q4[i] = fmaf(u.x, s[4 * i], fmaf(u.y, s[4 * i + 1], fmaf(u.z, s[4 * i + 2], u.w * s[4 * i + 3])));
      }
      float q = (q4[0] + q4[1]) + (q4[2] + q4[3]);
#pragma unroll
      for (int o = C::LPC / 2; o > 0; o >>= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
      float o4[4];
      const float4* pw = reinterpret_cast<const float4*>(s_w + j * DP) + l;
      const float4* pa = reinterpret_cast<const float4*>(s_a + j * DP) + l;
      const float4* pk = reinterpret_cast<const float4*>(s_k + j * DP) + l;
      const float4* pr = reinterpret_cast<const float4*>(s_r + j * DP) + l;
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const float4 w = pw[i * C::LPC], a = pa[i * C::LPC], k = pk[i * C::LPC], r = pr[i * C::LPC];
        s[4 * i] = fmaf(w.x, s[4 * i], fmaf(a.x, q, k.x * v));
        s[4 * i + 1] = fmaf(w.y, s[4 * i + 1], fmaf(a.y, q, k.y * v));
        s[4 * i + 2] = fmaf(w.z, s[4 * i + 2], fmaf(a.z, q, k.z * v));
        s[4 * i + 3] = fmaf(w.w, s[4 * i + 3], fmaf(a.w, q, k.w * v));
        o4[i] = fmaf(r.x, s[4 * i], fmaf(r.y, s[4 * i + 1], fmaf(r.z, s[4 * i + 2], r.w * s[4 * i + 3])));
      }
      float o = (o4[0] + o4[1]) + (o4[2] + o4[3]);
#pragma unroll
      for (int x = C::LPC / 2; x > 0; x >>= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
      if (l == 0 && col < p.dim) p.raw[((int64_t)b * p.S + t0 + j) * hd + head * p.dim + col] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < 16; i++) {
    const int k = (i >> 2) * 4 * C::LPC + l * 4 + (i & 3);
    if (col < p.dim && k < p.dim) st[(int64_t)k * p.dim] = s[i];
  }
}

// out = raw / rms(raw over the head) * norm_w * sigmoid(g): a warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) delta_out_kernel(const float* __restrict__ raw, const T* __restrict__ gate, const float* __restrict__ norm_w,
                                                        T* __restrict__ out, int64_t rows, int H, int dim, int64_t ldp, int64_t ldo, float eps) {
  pdl_trigger();
  pdl_wait();
  const int64_t item = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  const int64_t row = item / H;
  const int head = (int)(item % H);
  if (row >= rows) return;
  const float* x = raw + row * H * dim + head * dim;
  float ss = 0.0f;
  for (int i = lane; i < dim; i += 32) ss = fmaf(x[i], x[i], ss);
  const float inv = 1.0f / sqrtf(hy_warp_sum(ss) / (float)dim + eps);
  for (int i = lane; i < dim; i += 32) {
    const int c = head * dim + i;
    hy_st(out + row * ldo + c, x[i] * inv * norm_w[c] * hy_sigmoid(hy_ld(gate + row * ldp + c)));
  }
  if (head == H - 1)
    for (int64_t c = (int64_t)H * dim + lane; c < ldo; c += 32) hy_st(out + row * ldo + c, 0.0f);
}

template <typename T, int DP>
static int delta_launch(const DeltaParams<T>& p, cudaStream_t st) {
  using C = DeltaCfg<DP>;
  static bool opted[16] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (C::SMEM > 48 * 1024 && (dev < 0 || dev >= 16 || !opted[dev])) {
    TPX_CUDA_OK(cudaFuncSetAttribute(delta_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  TPX_CUDA_OK(launch_pdl(delta_kernel<T, DP>, dim3((unsigned)p.H, (unsigned)((p.dim + C::COLS - 1) / C::COLS), (unsigned)p.B), dim3(C::THREADS), C::SMEM,
                         st, p));
  return TPX_OK;
}

template <typename T>
static int delta_run(const TpxDeltaRule& a, cudaStream_t st) {
  DeltaParams<T> p = {(const T*)a.proj, a.wraw, a.a_bias, a.start, a.dev_len, a.state, a.raw, (int)a.B, (int)a.S, (int)a.past, (int)a.heads,
                      (int)a.dim, (long long)a.ldp};
  int rc;
  if (a.dim <= 32) rc = delta_launch<T, 32>(p, st);
  else if (a.dim <= 64) rc = delta_launch<T, 64>(p, st);
  else if (a.dim <= 128) rc = delta_launch<T, 128>(p, st);
  else if (a.dim <= 256) rc = delta_launch<T, 256>(p, st);
  else rc = delta_launch<T, 512>(p, st);
  if (rc) return rc;
  const int64_t rows = a.B * a.S, hd = a.heads * a.dim;
  TPX_CUDA_OK(launch_pdl(delta_out_kernel<T>, dim3((unsigned)((rows * a.heads + 7) / 8)), dim3(256), 0, st, (const float*)a.raw,
                         (const T*)a.proj + 4 * hd, a.norm_w, (T*)a.out, rows, (int)a.heads, (int)a.dim, a.ldp, a.ldo, a.eps));
  return TPX_OK;
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_delta_rule(const TpxDeltaRule* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "delta_rule: null argument block");
  TPX_REQUIRE(a->B >= 0 && a->S >= 0 && a->heads > 0 && a->dim > 0 && a->past >= 0, TPX_ERR_ARG, "delta_rule: bad shape");
  TPX_REQUIRE(a->dim <= 512, TPX_ERR_UNSUPPORTED, "delta_rule: heads of at most 512 channels, got %ld", (long)a->dim);
  TPX_REQUIRE(a->B <= 65535 && a->S < (1 << 24) && a->past < (1ll << 30) && a->heads < (1 << 16), TPX_ERR_ARG, "delta_rule: shape too large");
  if (a->B == 0 || a->S == 0) return TPX_OK;
  TPX_REQUIRE(a->proj && a->wraw && a->a_bias && a->norm_w && a->state && a->raw && a->out, TPX_ERR_ARG, "delta_rule: null pointer");
  TPX_REQUIRE(a->ldp >= 5 * a->heads * a->dim && a->ldo >= a->heads * a->dim, TPX_ERR_ARG, "delta_rule: a leading dimension is smaller than its row");
  TPX_REQUIRE(!a->dev_len || a->S == 1, TPX_ERR_ARG, "delta_rule: dev_len is for single tokens");
  return a->f32 ? delta_run<float>(*a, (cudaStream_t)stream) : delta_run<__nv_bfloat16>(*a, (cudaStream_t)stream);
}
