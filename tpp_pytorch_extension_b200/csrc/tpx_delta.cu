// Generalized delta rule (a linear recurrence with a matrix state per head), token by token in 32-bit:
//   S_t = diag(w_t) S_(t-1) - (a_t u_t)(u_t^T S_(t-1)) + k_t v_t^T,   o_t = S_t^T r_t,   u = k / sqrt(sum k^2 + 1e-6)
// A column of S (one value channel) evolves without the others: only the scalars u^T s and r^T s of the column are sums
// over key channels. So a CTA owns some columns of one (sequence, head); LPC = DP / 16 neighbouring lanes hold a column,
// 16 key channels each, in registers for the whole call. The vectors of 16 tokens at a time (decays, rates, unit keys: the
// exponentials and square roots) are prepared by all warps into shared memory.
// The read-outs go to `raw` in fp32; a second kernel divides each head by its root mean square and applies weight and gate.
//
// bf16 models with head sizes that are multiples of 8 up to 128 take delta_fast_kernel: one CTA per (sequence, head),
// DP / LPC key channels x CPT columns per thread, packed two-wide fp32 arithmetic, the next tokens' rows in flight
// (cp.async) while the current ones are worked on, output norm and gate in the same kernel. A vector element read from
// shared memory serves CPT columns, and shared memory gives 4 bytes per lane and cycle whatever the sharing between lanes:
// with four columns its loads take as long as the arithmetic, with eight half as long.
// Within a chunk of tokens the state is kept divided by the decay accumulated since the chunk's start, G:
//   S = G s,  s <- s - (a k / G_t) q + (k / G_t) v^T,  q = (G_(t-1) k)^T s / (sum k^2 + 1e-6),
//   o = (G_t r)^T s_(t-1) + (r . k) v - (r . a k) q
// so that a token costs four multiply-adds per state element instead of five and reads the state once; at the chunk's end
// s is multiplied by G. A decay is at least exp(-0.61), G at least 6e-5 after 16 tokens: nothing under- or overflows, and a
// scale per channel does not change relative rounding.
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

// ---------------------------------------------------------------- the bf16 kernel
__device__ __forceinline__ float2 dl_fma2(float2 a, float2 b, float2 c) {
  unsigned long long r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(r)
      : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)), "l"(*reinterpret_cast<unsigned long long*>(&c)));
  return *reinterpret_cast<float2*>(&r);
}
__device__ __forceinline__ float2 dl_mul2(float2 a, float2 b) {
  unsigned long long r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)));
  return *reinterpret_cast<float2*>(&r);
}
__device__ __forceinline__ void dl_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ float dl_sigmoid(float v) { return __fdividef(1.0f, 1.0f + __expf(-v)); }

struct DeltaFastParams {
  const uint16_t* proj;
  const float *wraw, *a_bias, *norm_w;
  const int *start, *dev_len;
  float* state;
  uint16_t* out;
  long long ldp, ldo;
  int S, past, H, dim;
  float eps;
};

template <int DP, int LPC, int CPT, int TC>
struct DfCfg {
  static constexpr int KPT = DP / LPC, THREADS = DP * LPC / CPT, NW = THREADS / 32;
  // floats: five staged vectors per token, the read-outs, G, three scalars per token
  static constexpr int STAGED = 6 * TC * DP + DP + 4 * TC;
  static constexpr int RAW = TC * DP * (5 * 2 + 4);  // bytes of one raw chunk: r, k, v, a, g in bf16, w in fp32
  static constexpr size_t SMEM = STAGED * 4 + 2 * RAW;
  static_assert(KPT % 4 == 0 && THREADS % 32 == 0 && LPC <= 32, "whole vectors and warps");
  static_assert(CPT == 2 || CPT % 4 == 0, "columns in pairs or fours");
};

template <int THREADS>
__device__ __forceinline__ void df_sync() {
  if (THREADS == 32) __syncwarp();
  else __syncthreads();
}

// EXACT: dim == DP, so that index arithmetic is by constants
template <int DP, int LPC, int CPT, int TC, bool EXACT>
__global__ void __launch_bounds__(DfCfg<DP, LPC, CPT, TC>::THREADS) delta_fast_kernel(DeltaFastParams p) {
  using C = DfCfg<DP, LPC, CPT, TC>;
  constexpr int KV = C::KPT / 4, KP = C::KPT / 2;  // float4 vectors, channel pairs per thread
  extern __shared__ __align__(16) float df_smem[];
  float *s_u = df_smem, *s_k = s_u + TC * DP, *s_a = s_k + TC * DP, *s_r = s_a + TC * DP, *s_v = s_r + TC * DP, *s_o = s_v + TC * DP;
  float* s_g = s_o + TC * DP;
  float4* s_sc = reinterpret_cast<float4*>(s_g + DP);  // per token: - 1 / (sum k^2 + 1e-6), r . k, r . (a k)
  unsigned char* raw = reinterpret_cast<unsigned char*>(s_sc + TC);
  pdl_trigger();
  const int head = blockIdx.x, b = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int l = tid % LPC, c0 = (tid / LPC) * CPT;
  const int dim = EXACT ? DP : p.dim, hd = p.H * dim;
  constexpr int CH = DP / 32;  // channels per lane when a warp works on a token
  float bias[CH], nw[CH];
#pragma unroll
  for (int i = 0; i < CH; i++) {
    const int c = lane + 32 * i;
    bias[i] = c < dim ? __ldg(p.a_bias + head * dim + c) : 0.0f;
    nw[i] = c < dim ? __ldg(p.norm_w + head * dim + c) : 0.0f;
  }
  pdl_wait();
  const int past = p.dev_len ? *p.dev_len : p.past;
  const int first = p.start ? max(0, min(p.S, p.start[b] - past)) : 0;
  const uint16_t* proj = p.proj + (long long)b * p.S * p.ldp + head * dim;
  const float* wraw = p.wraw + (long long)b * p.S * hd + head * dim;

  auto fetch = [&](int t0, int stage) {
    unsigned char* dst = raw + stage * C::RAW;
    const int n = min(TC, p.S - t0), dc = dim / 8;  // 16-byte units per bf16 row of a head
    for (int i = tid; i < n * 5 * dc; i += C::THREADS) {
      const int c = i % dc, a = (i / dc) % 5, t = i / (dc * 5);
      dl_cp16(dst + ((a * TC + t) * DP + c * 8) * 2, proj + (long long)(t0 + t) * p.ldp + a * hd + c * 8);
    }
    for (int i = tid; i < n * 2 * dc; i += C::THREADS) {
      const int c = i % (2 * dc), t = i / (2 * dc);
      dl_cp16(dst + 5 * TC * DP * 2 + (t * DP + c * 4) * 4, wraw + (long long)(t0 + t) * hd + c * 4);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (first < p.S) fetch(first, 0);

  float2 s[CPT][KP];  // [column][pair of key channels]
  float* st = p.state + (long long)(b * p.H + head) * dim * dim + c0;
#pragma unroll
  for (int i = 0; i < KP; i++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int k = (i >> 1) * 4 * LPC + l * 4 + (i & 1) * 2 + e;
      if constexpr (CPT % 4 == 0) {
#pragma unroll
        for (int c = 0; c < CPT; c += 4) {
          const float4 v = (k < dim && c0 + c < dim) ? *reinterpret_cast<const float4*>(st + (long long)k * dim + c) : make_float4(0, 0, 0, 0);
          const float vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
          for (int d = 0; d < 4; d++) {
            if (e) s[c + d][i].y = vv[d];
            else s[c + d][i].x = vv[d];
          }
        }
      } else {
        const int c = 0;
        const float2 v = (k < dim && c0 + c < dim) ? *reinterpret_cast<const float2*>(st + (long long)k * dim + c) : make_float2(0, 0);
        if (e) { s[c][i].y = v.x; s[c + 1][i].y = v.y; }
        else { s[c][i].x = v.x; s[c + 1][i].x = v.y; }
      }
    }

  int stage = 0;
  for (int t0 = first; t0 < p.S; t0 += TC, stage ^= 1) {
    const int n = min(TC, p.S - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    df_sync<C::THREADS>();
    if (t0 + TC < p.S) fetch(t0 + TC, stage ^ 1);
    const uint16_t* rb = reinterpret_cast<const uint16_t*>(raw + stage * C::RAW);
    const float* rw = reinterpret_cast<const float*>(raw + stage * C::RAW + 5 * TC * DP * 2);
    // decays, rates and the tokens' scalars: a warp per token; tokens beyond the call's last one leave the state as it is
#pragma unroll 2
    for (int t = warp; t < TC; t += C::NW) {
      float k2 = 0.0f, rk = 0.0f, ra = 0.0f;
#pragma unroll
      for (int i = 0; i < CH; i++) {
        const int c = lane + 32 * i;
        float r = 0, k = 0, v = 0, ak = 0, w = 1.0f;
        if (c < dim && t < n) {
          r = bf16_bits_to_f32(rb[(0 * TC + t) * DP + c]);
          k = bf16_bits_to_f32(rb[(1 * TC + t) * DP + c]);
          v = bf16_bits_to_f32(rb[(2 * TC + t) * DP + c]);
          ak = dl_sigmoid(bf16_bits_to_f32(rb[(3 * TC + t) * DP + c]) + bias[i]) * k;
          w = __expf(-0.60653065971263342f * dl_sigmoid(rw[t * DP + c]));
        }
        k2 = fmaf(k, k, k2);
        rk = fmaf(r, k, rk);
        ra = fmaf(r, ak, ra);
        s_u[t * DP + c] = w;
        s_k[t * DP + c] = k;
        s_a[t * DP + c] = ak;
        s_r[t * DP + c] = r;
        s_v[t * DP + c] = v;
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        k2 += __shfl_xor_sync(0xffffffffu, k2, o);
        rk += __shfl_xor_sync(0xffffffffu, rk, o);
        ra += __shfl_xor_sync(0xffffffffu, ra, o);
      }
      if (lane == 0) s_sc[t] = make_float4(-1.0f / (k2 + 1e-6f), rk, ra, 0.0f);
    }
    df_sync<C::THREADS>();
    // accumulated decays: a thread per channel, all loads ahead of the stores
    for (int c = tid; c < DP; c += C::THREADS) {
      float w[TC], k[TC], ak[TC], r[TC];
#pragma unroll
      for (int t = 0; t < TC; t++) { w[t] = s_u[t * DP + c]; k[t] = s_k[t * DP + c]; ak[t] = s_a[t * DP + c]; r[t] = s_r[t * DP + c]; }
      float g = 1.0f;
#pragma unroll
      for (int t = 0; t < TC; t++) {
        s_u[t * DP + c] = g * k[t];
        g *= w[t];
        const float gi = __fdividef(1.0f, g);
        s_k[t * DP + c] = k[t] * gi;
        s_a[t * DP + c] = ak[t] * gi;
        s_r[t * DP + c] = r[t] * g;
      }
      s_g[c] = g;
    }
    df_sync<C::THREADS>();
    const uint32_t so = (uint32_t)__cvta_generic_to_shared(s_o);
    constexpr int UNROLL = TC < 4 ? TC : 4;
#pragma unroll UNROLL
    for (int t = 0; t < TC; t++) {
      const float4* pu = reinterpret_cast<const float4*>(s_u + t * DP) + l;
      const float4* pr = reinterpret_cast<const float4*>(s_r + t * DP) + l;
      float2 qa[CPT], oa[CPT];
#pragma unroll
      for (int c = 0; c < CPT; c++) qa[c] = oa[c] = make_float2(0.0f, 0.0f);
      float v[CPT];
      if constexpr (CPT % 4 == 0) {
#pragma unroll
        for (int c = 0; c < CPT; c += 4) {
          const float4 x = *reinterpret_cast<const float4*>(s_v + t * DP + c0 + c);
          v[c] = x.x; v[c + 1] = x.y; v[c + 2] = x.z; v[c + 3] = x.w;
        }
      } else {
        const float2 x = *reinterpret_cast<const float2*>(s_v + t * DP + c0);
        v[0] = x.x; v[1] = x.y;
      }
#pragma unroll
      for (int i = 0; i < KV; i++) {
        const float4 u = pu[i * LPC];
#pragma unroll
        for (int c = 0; c < CPT; c++) {
          qa[c] = dl_fma2(make_float2(u.x, u.y), s[c][2 * i], qa[c]);
          qa[c] = dl_fma2(make_float2(u.z, u.w), s[c][2 * i + 1], qa[c]);
        }
      }
      float q[CPT], o[CPT];
#pragma unroll
      for (int c = 0; c < CPT; c++) q[c] = qa[c].x + qa[c].y;
#pragma unroll
      for (int x = LPC / 2; x > 0; x >>= 1)
#pragma unroll
        for (int c = 0; c < CPT; c++) q[c] += __shfl_xor_sync(0xffffffffu, q[c], x);
#pragma unroll
      for (int i = 0; i < KV; i++) {  // independent of q: fills the time of the shuffles
        const float4 r = pr[i * LPC];
#pragma unroll
        for (int c = 0; c < CPT; c++) {
          oa[c] = dl_fma2(make_float2(r.x, r.y), s[c][2 * i], oa[c]);
          oa[c] = dl_fma2(make_float2(r.z, r.w), s[c][2 * i + 1], oa[c]);
        }
      }
      const float4 sc = s_sc[t];
      const float rk = l == 0 ? sc.y : 0.0f, ra = l == 0 ? sc.z : 0.0f;  // one lane of a column adds the scalar terms
      const float4* pk = reinterpret_cast<const float4*>(s_k + t * DP) + l;
      const float4* pa = reinterpret_cast<const float4*>(s_a + t * DP) + l;
#pragma unroll
      for (int c = 0; c < CPT; c++) {
        q[c] *= sc.x;
        o[c] = fmaf(rk, v[c], fmaf(ra, q[c], oa[c].x + oa[c].y));
      }
#pragma unroll
      for (int i = 0; i < KV; i++) {
        const float4 k = pk[i * LPC], a = pa[i * LPC];
#pragma unroll
        for (int c = 0; c < CPT; c++) {
          const float2 vv = make_float2(v[c], v[c]), qq = make_float2(q[c], q[c]);
          s[c][2 * i] = dl_fma2(make_float2(a.x, a.y), qq, dl_fma2(make_float2(k.x, k.y), vv, s[c][2 * i]));
          s[c][2 * i + 1] = dl_fma2(make_float2(a.z, a.w), qq, dl_fma2(make_float2(k.z, k.w), vv, s[c][2 * i + 1]));
        }
      }
      // sum over the column's lanes, every step leaving a lane half of its columns: lane l ends with columns l * CPT / LPC ...
      constexpr int LEFT = CPT > LPC ? CPT / LPC : 1, SKIP = LPC > CPT ? LPC / CPT : 1;
#pragma unroll
      for (int x = LPC / 2, m = CPT; x > 0; x >>= 1) {
        if (m > 1) {
          m >>= 1;
          const bool up = (l & x) != 0;
#pragma unroll
          for (int c = 0; c < CPT / 2; c++)
            if (c < m) {
              const float mine = up ? o[c + m] : o[c], other = up ? o[c] : o[c + m];
              o[c] = mine + __shfl_xor_sync(0xffffffffu, other, x);
            }
        } else {
          o[0] += __shfl_xor_sync(0xffffffffu, o[0], x);
        }
      }
      // stored without a memory clobber: nothing but the next barrier orders these against other accesses, so that the next
      // token's loads may move ahead of them
      if (l % SKIP == 0)
#pragma unroll
        for (int c = 0; c < LEFT; c++)
          asm volatile("st.shared.f32 [%0], %1;" ::"r"(so + (uint32_t)(t * DP + c0 + l * CPT / LPC + c) * 4), "f"(o[c]));
    }
    {
      const float4* pg = reinterpret_cast<const float4*>(s_g) + l;
#pragma unroll
      for (int i = 0; i < KV; i++) {
        const float4 g = pg[i * LPC];
#pragma unroll
        for (int c = 0; c < CPT; c++) {
          s[c][2 * i] = dl_mul2(make_float2(g.x, g.y), s[c][2 * i]);
          s[c][2 * i + 1] = dl_mul2(make_float2(g.z, g.w), s[c][2 * i + 1]);
        }
      }
    }
    asm volatile("" ::: "memory");
    df_sync<C::THREADS>();
    // output norm and gate: a warp per token
#pragma unroll 2
    for (int t = warp; t < n; t += C::NW) {
      float x[CH], ss = 0.0f;
#pragma unroll
      for (int i = 0; i < CH; i++) {
        x[i] = lane + 32 * i < dim ? s_o[t * DP + lane + 32 * i] : 0.0f;
        ss = fmaf(x[i], x[i], ss);
      }
      const float inv = rsqrtf(hy_warp_sum(ss) / (float)dim + p.eps);
      uint16_t* out = p.out + ((long long)b * p.S + t0 + t) * p.ldo + head * dim;
#pragma unroll
      for (int i = 0; i < CH; i++)
        if (lane + 32 * i < dim)
          out[lane + 32 * i] = f32_to_bf16_bits(x[i] * inv * nw[i] * dl_sigmoid(bf16_bits_to_f32(rb[(4 * TC + t) * DP + lane + 32 * i])));
    }
  }
#pragma unroll
  for (int i = 0; i < KP; i++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int k = (i >> 1) * 4 * LPC + l * 4 + (i & 1) * 2 + e;
      if constexpr (CPT % 4 == 0) {
#pragma unroll
        for (int c = 0; c < CPT; c += 4)
          if (k < dim && c0 + c < dim)
            *reinterpret_cast<float4*>(st + (long long)k * dim + c) =
                e ? make_float4(s[c][i].y, s[c + 1][i].y, s[c + 2][i].y, s[c + 3][i].y) : make_float4(s[c][i].x, s[c + 1][i].x, s[c + 2][i].x, s[c + 3][i].x);
      } else {
        const int c = 0;
        if (k < dim && c0 < dim)
          *reinterpret_cast<float2*>(st + (long long)k * dim + c) = e ? make_float2(s[c][i].y, s[c + 1][i].y) : make_float2(s[c][i].x, s[c + 1][i].x);
      }
    }
}

template <int DP, int LPC, int CPT, int TC>
static int delta_fast_launch(const DeltaFastParams& p, int64_t B, cudaStream_t st) {
  using C = DfCfg<DP, LPC, CPT, TC>;
  void (*k)(DeltaFastParams) = p.dim == DP ? delta_fast_kernel<DP, LPC, CPT, TC, true> : delta_fast_kernel<DP, LPC, CPT, TC, false>;
  static bool opted[16] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (C::SMEM > 48 * 1024 && (dev < 0 || dev >= 16 || !opted[dev])) {
    TPX_CUDA_OK(cudaFuncSetAttribute(delta_fast_kernel<DP, LPC, CPT, TC, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    TPX_CUDA_OK(cudaFuncSetAttribute(delta_fast_kernel<DP, LPC, CPT, TC, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)p.H, (unsigned)B), dim3(C::THREADS), C::SMEM, st, p));
  return TPX_OK;
}

static bool delta_fast_serves(const TpxDeltaRule& a) {
  return !a.f32 && a.dim % 8 == 0 && a.dim <= 128 && a.ldp % 8 == 0 && a.ldo == a.heads * a.dim &&
         (((uintptr_t)a.proj | (uintptr_t)a.wraw | (uintptr_t)a.out | (uintptr_t)a.norm_w | (uintptr_t)a.state) & 15) == 0;
}

static int delta_fast(const TpxDeltaRule& a, cudaStream_t st) {
  DeltaFastParams p = {(const uint16_t*)a.proj, a.wraw, a.a_bias, a.norm_w, a.start, a.dev_len, a.state, (uint16_t*)a.out, (long long)a.ldp,
                       (long long)a.ldo, (int)a.S, (int)a.past, (int)a.heads, (int)a.dim, a.eps};
  // eight columns per thread and few warps per head when there are many heads, more warps per head when a token's latency counts
  const bool many = a.B * a.heads >= (a.dim <= 64 ? 4 : 2) * sm_count();
  if (a.dim <= 32) return a.S == 1 ? delta_fast_launch<32, 4, 4, 1>(p, a.B, st) : delta_fast_launch<32, 4, 4, 8>(p, a.B, st);
  if (a.dim <= 64) {
    if (a.S == 1) return delta_fast_launch<64, 8, 4, 1>(p, a.B, st);
    if (many) return delta_fast_launch<64, 4, 8, 8>(p, a.B, st);
    return a.B * a.heads > sm_count() ? delta_fast_launch<64, 8, 4, 16>(p, a.B, st) : delta_fast_launch<64, 8, 2, 16>(p, a.B, st);
  }
  if (a.S == 1) return delta_fast_launch<128, 16, 4, 1>(p, a.B, st);
  return many ? delta_fast_launch<128, 8, 8, 8>(p, a.B, st) : delta_fast_launch<128, 8, 4, 8>(p, a.B, st);
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
  if (delta_fast_serves(*a)) return delta_fast(*a, (cudaStream_t)stream);
  return a->f32 ? delta_run<float>(*a, (cudaStream_t)stream) : delta_run<__nv_bfloat16>(*a, (cudaStream_t)stream);
}
