// Gated linear attention: per head a matrix state S [dim][vdim] with a decay per key channel,
//   S_t = diag(w_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t dim^(-1/2),   w = sigmoid(z)^(1/tau)
// then each head's o over its root mean square, times a weight, times silu of its gate. Everything between the projections and
// the output is 32-bit.
//
// A column of S (one value channel) evolves without the others, so the work can be cut along value channels; only the output
// norm needs a whole head. Kernels:
//   gla_fast_kernel   bf16, several tokens. Tokens go through the state four at a time: with c_t the decays' product from
//                     the block's first token to t, and s_t that from t + 1 to its last,
//                       o_t = (q_t c_t)^T S + sum_(u <= t) (q_t . k_u prod_(u < x <= t) w_x) v_u,
//                       S <- diag(c_3) S + sum_t (k_t s_t) v_t^T
//                     i.e. 9 operations per state element for four tokens instead of 12, no division by a decay (all factors are
//                     products of decays, at most 1), and no dependency between lanes. The state stays in registers, in pairs of key channels
//                     (packed fp32). DP / LPC key channels x CPT columns per thread.
//   gla_token_kernel  one token: a CTA per (sequence, head) streams the state through once; the low-rank map of the decay is
//                     computed here as well.
//   gla_kernel        any type and size, token by token; a column's key channels on neighbouring lanes.
// The last and the column-cut form of the first leave o in `raw`; gla_out_kernel finishes it.
#include "tpx_hybrid.cuh"

namespace tpx {

// sigmoid(z)^(1/tau)
__device__ __forceinline__ float gla_decay(float z, float inv_tau) {
  const float softplus = fmaxf(-z, 0.0f) + log1pf(expf(-fabsf(z)));
  return expf(-softplus * inv_tau);
}
__device__ __forceinline__ float gla_silu(float g) { return g * hy_sigmoid(g); }
__device__ __forceinline__ int gla_first(const TpxGla& p, int b) {  // tokens of this call that are padding
  if (!p.start) return 0;
  const int64_t past = p.dev_len ? *p.dev_len : p.past, n = p.start[b] - past;
  return n < 0 ? 0 : n > p.S ? (int)p.S : (int)n;
}

// ---------------------------------------------------------------- any type and size
constexpr int kGlaTok = 8;

template <int DP>
struct GlaCfg {
  static constexpr int LPC = DP / 16, COLS = 128 / LPC, THREADS = 128;
  static constexpr size_t SMEM = (size_t)kGlaTok * (3 * DP + COLS) * 4;
};

template <typename T, int DP>
__global__ void __launch_bounds__(128) gla_kernel(TpxGla p) {
  using C = GlaCfg<DP>;
  extern __shared__ __align__(16) float gl_smem[];
  float *s_w = gl_smem, *s_k = s_w + kGlaTok * DP, *s_q = s_k + kGlaTok * DP, *s_v = s_q + kGlaTok * DP;
  pdl_trigger();
  pdl_wait();
  const int head = blockIdx.x, c0 = blockIdx.y * C::COLS, b = blockIdx.z;
  const int l = threadIdx.x % C::LPC, cl = threadIdx.x / C::LPC, col = c0 + cl;
  const int dim = (int)p.dim, vdim = (int)p.vdim, S = (int)p.S;
  const float scale = 1.0f / sqrtf((float)dim), inv_tau = 1.0f / p.tau;
  float* st = p.state + ((int64_t)(b * p.heads + head) * dim) * vdim + col;
  float s[16];
#pragma unroll
  for (int i = 0; i < 16; i++) {
    const int k = i * C::LPC + l;
    s[i] = (col < vdim && k < dim) ? st[(int64_t)k * vdim] : 0.0f;
  }
  for (int t0 = gla_first(p, b); t0 < S; t0 += kGlaTok) {
    const int n = min(kGlaTok, S - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < n * DP; i += 128) {
      const int j = i / DP, c = i % DP;
      const int64_t row = (int64_t)b * S + t0 + j;
      const T* pr = reinterpret_cast<const T*>(p.proj) + row * p.ldp + (int64_t)head * dim + c;
      const bool in = c < dim;
      s_w[i] = in ? gla_decay(p.zraw[(row * p.heads + head) * dim + c], inv_tau) : 0.0f;
      s_k[i] = in ? hy_ld(pr + p.k_col) : 0.0f;
      s_q[i] = in ? hy_ld(pr + p.q_col) * scale : 0.0f;
    }
    for (int i = threadIdx.x; i < n * C::COLS; i += 128) {
      const int j = i / C::COLS, c = c0 + i % C::COLS;
      s_v[i] = c < vdim ? hy_ld(reinterpret_cast<const T*>(p.proj) + ((int64_t)b * S + t0 + j) * p.ldp + p.v_col + (int64_t)head * vdim + c) : 0.0f;
    }
    __syncthreads();
    for (int j = 0; j < n; j++) {
      const float v = s_v[j * C::COLS + cl];
      float o = 0.0f;
#pragma unroll
      for (int i = 0; i < 16; i++) {
        const int k = j * DP + i * C::LPC + l;
        s[i] = fmaf(s_w[k], s[i], s_k[k] * v);
        o = fmaf(s_q[k], s[i], o);
      }
#pragma unroll
      for (int x = C::LPC / 2; x > 0; x >>= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
      if (l == 0 && col < vdim) p.raw[(((int64_t)b * S + t0 + j) * p.heads + head) * vdim + col] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < 16; i++) {
    const int k = i * C::LPC + l;
    if (col < vdim && k < dim) st[(int64_t)k * vdim] = s[i];
  }
}

// out = raw / rms(raw over the head) * norm_w * silu(g), zero for padding: a warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) gla_out_kernel(TpxGla p) {
  pdl_trigger();
  pdl_wait();
  const int64_t item = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, vdim = (int)p.vdim;
  const int64_t row = item / p.heads;
  const int head = (int)(item % p.heads);
  if (row >= p.B * p.S) return;
  const bool pad = row % p.S < gla_first(p, (int)(row / p.S));
  const float* x = p.raw + item * vdim;
  const T* g = reinterpret_cast<const T*>(p.proj) + row * p.ldp + p.g_col + (int64_t)head * vdim;
  T* out = reinterpret_cast<T*>(p.out) + row * p.ldo + (int64_t)head * vdim;
  float ss = 0.0f;
  for (int i = lane; i < vdim; i += 32) ss = fmaf(x[i], x[i], ss);
  const float inv = 1.0f / sqrtf(hy_warp_sum(ss) / (float)vdim + p.eps);
  for (int i = lane; i < vdim; i += 32) hy_st(out + i, pad ? 0.0f : x[i] * inv * p.norm_w[i] * gla_silu(hy_ld(g + i)));
}

// ---------------------------------------------------------------- one token
// 256 threads: vdim / 4 groups of four columns x rows; ROWS state rows per thread and pass
constexpr int kGlaTokThreads = 256, kGlaTokRows = 8;

template <typename T>
__global__ void __launch_bounds__(kGlaTokThreads) gla_token_kernel(TpxGla p) {
  extern __shared__ __align__(16) float gt_smem[];
  __shared__ float red[32];
  const int dim = (int)p.dim, vdim = (int)p.vdim, rank = (int)p.rank;
  const int ncg = vdim / 4, nrg = kGlaTokThreads / ncg;
  const int cg = threadIdx.x % ncg, rg = threadIdx.x / ncg;
  const bool live = rg < nrg;
  float *s_w = gt_smem, *s_k = s_w + dim, *s_q = s_k + dim;
  float4* s_o = reinterpret_cast<float4*>(s_q + dim + (-3 * dim & 3));  // [nrg][ncg]
  pdl_trigger();
  pdl_wait();
  const int head = blockIdx.x, b = blockIdx.y;
  const T* pr = reinterpret_cast<const T*>(p.proj) + (int64_t)b * p.ldp;
  T* out = reinterpret_cast<T*>(p.out) + (int64_t)b * p.ldo + (int64_t)head * vdim;
  if (gla_first(p, b)) {
    for (int c = threadIdx.x; c < vdim; c += kGlaTokThreads) hy_st(out + c, 0.0f);
    return;
  }
  float4* st = reinterpret_cast<float4*>(p.state + ((int64_t)(b * p.heads + head) * dim) * vdim) + cg;
  float4 s[kGlaTokRows];
  auto load = [&](int r0) {
#pragma unroll
    for (int i = 0; i < kGlaTokRows; i++) {
      const int r = r0 + i * nrg;
      s[i] = live && r < dim ? st[(int64_t)r * ncg] : make_float4(0, 0, 0, 0);
    }
  };
  load(rg);
  const float scale = 1.0f / sqrtf((float)dim), inv_tau = 1.0f / p.tau;
  for (int c = threadIdx.x; c < dim; c += kGlaTokThreads) {
    const int64_t hc = (int64_t)head * dim + c;
    float z;
    if (p.zraw) {
      z = p.zraw[(int64_t)b * p.heads * dim + hc];
    } else {
      z = p.a2_bias[hc];
      const T* w = reinterpret_cast<const T*>(p.a2) + hc * p.lda2;
      for (int r = 0; r < rank; r++) z = fmaf(hy_ld(w + r), hy_ld(pr + p.a1_col + r), z);
    }
    s_w[c] = gla_decay(z, inv_tau);
    s_k[c] = hy_ld(pr + p.k_col + hc);
    s_q[c] = hy_ld(pr + p.q_col + hc) * scale;
  }
  float v[4] = {};
  if (live)
#pragma unroll
    for (int e = 0; e < 4; e++) v[e] = hy_ld(pr + p.v_col + (int64_t)head * vdim + cg * 4 + e);
  __syncthreads();
  float4 o = make_float4(0, 0, 0, 0);
  for (int r0 = rg; r0 < dim; r0 += nrg * kGlaTokRows) {
    if (r0 != rg) load(r0);
#pragma unroll
    for (int i = 0; i < kGlaTokRows; i++) {
      const int r = r0 + i * nrg;
      if (live && r < dim) {
        const float w = s_w[r], k = s_k[r], q = s_q[r];
        float4 x = s[i];
        x.x = fmaf(w, x.x, k * v[0]); x.y = fmaf(w, x.y, k * v[1]); x.z = fmaf(w, x.z, k * v[2]); x.w = fmaf(w, x.w, k * v[3]);
        st[(int64_t)r * ncg] = x;
        o.x = fmaf(q, x.x, o.x); o.y = fmaf(q, x.y, o.y); o.z = fmaf(q, x.z, o.z); o.w = fmaf(q, x.w, o.w);
      }
    }
  }
  if (live) s_o[rg * ncg + cg] = o;
  __syncthreads();
  // columns in the order of the threads: thread c sums column c, c + 256, ...
  const float* so = reinterpret_cast<const float*>(s_o);
  float x[4], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int c = threadIdx.x + i * kGlaTokThreads;
    x[i] = 0.0f;
    if (c < vdim)
      for (int r = 0; r < nrg; r++) x[i] += so[r * vdim + c];
    ss = fmaf(x[i], x[i], ss);
  }
  const float inv = 1.0f / sqrtf(hy_block_sum(ss, red) / (float)vdim + p.eps);
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int c = threadIdx.x + i * kGlaTokThreads;
    if (c < vdim) hy_st(out + c, x[i] * inv * p.norm_w[c] * gla_silu(hy_ld(pr + p.g_col + (int64_t)head * vdim + c)));
  }
}

// ---------------------------------------------------------------- bf16, several tokens
// the same on the special-function unit; what counts of the logarithm is its absolute error, below 4e-7
__device__ __forceinline__ float gl_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gl_decay(float z, float inv_tau) {
  const float y = z * -1.4426950408889634f;
  float lg;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(lg) : "f"(1.0f + gl_ex2(-fabsf(y))));
  return gl_ex2((fmaxf(y, 0.0f) + lg) * -inv_tau);
}
__device__ __forceinline__ float gl_silu(float g) { return __fdividef(g, 1.0f + __expf(-g)); }
__device__ __forceinline__ float2 gl_fma2(float2 a, float2 b, float2 c) {
  unsigned long long r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(r)
      : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)), "l"(*reinterpret_cast<unsigned long long*>(&c)));
  return *reinterpret_cast<float2*>(&r);
}
__device__ __forceinline__ float2 gl_mul2(float2 a, float2 b) {
  unsigned long long r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)));
  return *reinterpret_cast<float2*>(&r);
}
__device__ __forceinline__ void gl_cp16(void* dst, const void* src, bool ok) {  // zeros unless ok
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ float gl_lo(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float gl_hi(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }
// N consecutive bf16 values from shared memory as floats
template <int N>
__device__ __forceinline__ void gl_ld_bf16(const uint16_t* p, float (&v)[N]) {
  if constexpr (N % 8 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 8) {
      const uint4 u = *reinterpret_cast<const uint4*>(p + i);
      v[i] = gl_lo(u.x); v[i + 1] = gl_hi(u.x); v[i + 2] = gl_lo(u.y); v[i + 3] = gl_hi(u.y);
      v[i + 4] = gl_lo(u.z); v[i + 5] = gl_hi(u.z); v[i + 6] = gl_lo(u.w); v[i + 7] = gl_hi(u.w);
    }
  } else if constexpr (N == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    v[0] = gl_lo(u.x); v[1] = gl_hi(u.x); v[2] = gl_lo(u.y); v[3] = gl_hi(u.y);
  } else if constexpr (N == 2) {
    const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
    v[0] = gl_lo(u); v[1] = gl_hi(u);
  } else {
    static_assert(N == 1, "vector size");
    v[0] = bf16_bits_to_f32(*p);
  }
}

template <int N>
__device__ __forceinline__ void gl_ld_f32(const float* p, float (&v)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      const float4 u = *reinterpret_cast<const float4*>(p + i);
      v[i] = u.x; v[i + 1] = u.y; v[i + 2] = u.z; v[i + 3] = u.w;
    }
  } else if constexpr (N == 2) {
    const float2 u = *reinterpret_cast<const float2*>(p);
    v[0] = u.x; v[1] = u.y;
  } else {
    static_assert(N == 1, "vector size");
    v[0] = *p;
  }
}
template <int N>
__device__ __forceinline__ void gl_st_f32(float* p, const float (&v)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else if constexpr (N == 2) {
    *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  } else {
    static_assert(N == 1, "vector size");
    *p = v[0];
  }
}

// DP: key channels (padded), EC: columns of a CTA, LPC lanes per column, CPT columns per thread, TC tokens staged at once;
// WHOLE: the CTA has all columns of the head and finishes the output
template <int DP, int EC, int LPC, int CPT, int TC, bool WHOLE>
struct GfCfg {
  static constexpr int KPT = DP / LPC, THREADS = EC / CPT * LPC, NW = THREADS / 32, NB = TC / 4;
  static constexpr int STAGED = 2 * TC * DP + NB * (DP + 16) + (WHOLE ? TC * EC : 0);  // floats
  static constexpr int RQ = 0, RK = TC * DP * 2, RZ = 2 * RK, RV = RZ + TC * DP * 4, RG = RV + TC * EC * 2, RAW = RG + (WHOLE ? TC * EC * 2 : 0);
  static constexpr size_t SMEM = STAGED * 4 + 2 * RAW;
  static constexpr int M = 4 * CPT / LPC;  // read-outs a lane ends with per block of four tokens
  static_assert(KPT % 4 == 0 && THREADS % 32 == 0 && LPC <= 32 && 4 * CPT >= LPC && (STAGED * 4) % 16 == 0, "whole vectors and warps");
  static_assert(M <= CPT, "a lane's read-outs belong to one token");
  // 16-byte units that a thread copies: rows of DP bf16, DP fp32, EC bf16; a thread keeps its place in the row
  static constexpr int UD = DP / 8, UZ = DP / 4, UE = EC / 8;
  static_assert(THREADS % UD == 0 && THREADS % UZ == 0 && THREADS % UE == 0, "copies");
  static constexpr int OW = EC / 32;  // columns per lane in the output norm
};

template <int THREADS>
__device__ __forceinline__ void gl_sync() {
  if (THREADS == 32) __syncwarp();
  else __syncthreads();
}

template <int DP, int EC, int LPC, int CPT, int TC, bool WHOLE>
__global__ void __launch_bounds__(GfCfg<DP, EC, LPC, CPT, TC, WHOLE>::THREADS) gla_fast_kernel(TpxGla p) {
  using C = GfCfg<DP, EC, LPC, CPT, TC, WHOLE>;
  constexpr int KV = C::KPT / 4, KP = C::KPT / 2, M = C::M;
  extern __shared__ __align__(16) float gf_smem[];
  float *s_q = gf_smem, *s_k = s_q + TC * DP, *s_a = s_k + TC * DP, *s_d = s_a + C::NB * DP, *s_o = s_d + C::NB * 16;
  unsigned char* raw = reinterpret_cast<unsigned char*>(gf_smem + C::STAGED);
  pdl_trigger();
  const int head = blockIdx.x, b = blockIdx.z, e0 = blockIdx.y * EC;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int l = tid % LPC, c0 = (tid / LPC) * CPT;
  const int dim = (int)p.dim, vdim = (int)p.vdim, S = (int)p.S, ldp = (int)p.ldp, zd = (int)p.heads * dim;
  const int cols = min(EC, vdim - e0);
  const float scale = 1.0f / sqrtf((float)dim), inv_tau = 1.0f / p.tau;
  constexpr int CW = DP / 32;  // channels per lane where a warp has the whole head
  pdl_wait();
  const int first = gla_first(p, b);
  const int64_t row0 = (int64_t)b * S;
  const uint16_t* proj = reinterpret_cast<const uint16_t*>(p.proj) + (row0 + first) * ldp;
  // this thread's places in the rows it copies
  const uint16_t* fq = proj + (int64_t)(tid / C::UD) * ldp + p.q_col + head * dim + tid % C::UD * 8;
  const uint16_t* fv = proj + (int64_t)(tid / C::UE) * ldp + p.v_col + head * vdim + e0 + tid % C::UE * 8;
  const float* fz = p.zraw + (row0 + first + tid / C::UZ) * zd + head * dim + tid % C::UZ * 4;
  const int64_t kq = p.k_col - p.q_col, gv = p.g_col - p.v_col;
  const bool inq = tid % C::UD * 8 < dim, inz = tid % C::UZ * 4 < dim, inv = tid % C::UE * 8 < cols;

  auto fetch = [&](int t0, int stage) {  // tokens beyond the call and channels beyond the head read as zero
    unsigned char* dst = raw + stage * C::RAW + tid * 16;
    const int n = S - t0;
#pragma unroll
    for (int i = 0; i < TC; i += C::THREADS / C::UD) {
      const bool ok = inq && tid / C::UD + i < n && (C::THREADS / C::UD <= TC || tid / C::UD < TC);
      const uint16_t* src = ok ? fq + (int64_t)i * ldp : proj;
      if (C::THREADS / C::UD <= TC || tid / C::UD < TC) {
        gl_cp16(dst + C::RQ + i * DP * 2, src, ok);
        gl_cp16(dst + C::RK + i * DP * 2, ok ? src + kq : proj, ok);
      }
    }
#pragma unroll
    for (int i = 0; i < TC; i += C::THREADS / C::UZ) {
      const bool ok = inz && tid / C::UZ + i < n;
      if (C::THREADS / C::UZ <= TC || tid / C::UZ < TC) gl_cp16(dst + C::RZ + i * DP * 4, ok ? (const void*)(fz + (int64_t)i * zd) : proj, ok);
    }
#pragma unroll
    for (int i = 0; i < TC; i += C::THREADS / C::UE) {
      const bool ok = inv && tid / C::UE + i < n;
      const uint16_t* src = ok ? fv + (int64_t)i * ldp : proj;
      if (C::THREADS / C::UE <= TC || tid / C::UE < TC) {
        gl_cp16(dst + C::RV + i * EC * 2, src, ok);
        if (WHOLE) gl_cp16(dst + C::RG + i * EC * 2, ok ? src + gv : proj, ok);
      }
    }
    fq += (int64_t)TC * ldp;
    fv += (int64_t)TC * ldp;
    fz += (int64_t)TC * zd;
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (first < S) fetch(first, 0);
  if (WHOLE) {  // padding
    uint16_t* out = reinterpret_cast<uint16_t*>(p.out) + row0 * p.ldo + head * vdim;
    for (int i = tid; i < first * vdim; i += C::THREADS) out[(int64_t)(i / vdim) * p.ldo + i % vdim] = 0;
  }

  float nw[WHOLE ? C::OW : 1];
  if (WHOLE)
#pragma unroll
    for (int i = 0; i < C::OW; i++) nw[i] = lane * C::OW + i < vdim ? __ldg(p.norm_w + lane * C::OW + i) : 0.0f;
  float2 s[CPT][KP];  // [column][pair of key channels]
  float* st = p.state + ((int64_t)(b * p.heads + head) * dim) * vdim + e0 + c0;
#pragma unroll
  for (int i = 0; i < KP; i++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int k = (i >> 1) * 4 * LPC + l * 4 + (i & 1) * 2 + e;
#pragma unroll
      for (int c = 0; c < CPT; c += 4) {
        const float4 v = (k < dim && c0 + c < cols) ? *reinterpret_cast<const float4*>(st + (int64_t)k * vdim + c) : make_float4(0, 0, 0, 0);
        const float vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int d = 0; d < 4; d++) {
          if (e) s[c + d][i].y = vv[d];
          else s[c + d][i].x = vv[d];
        }
      }
    }

  int stage = 0;
  for (int t0 = first; t0 < S; t0 += TC, stage ^= 1) {
    const int n = min(TC, S - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    gl_sync<C::THREADS>();
    if (t0 + TC < S) fetch(t0 + TC, stage ^ 1);
    const unsigned char* rw = raw + stage * C::RAW;
    const uint16_t* rv = reinterpret_cast<const uint16_t*>(rw + C::RV);
    // the vectors of a block of four tokens: a warp per block, neighbouring channels per lane
    for (int blk = warp; blk < C::NB; blk += C::NW) {
      const int c = lane * CW;
      const uint16_t* rq = reinterpret_cast<const uint16_t*>(rw + C::RQ) + blk * 4 * DP + c;
      const uint16_t* rk = reinterpret_cast<const uint16_t*>(rw + C::RK) + blk * 4 * DP + c;
      const float* rz = reinterpret_cast<const float*>(rw + C::RZ) + blk * 4 * DP + c;
      float q[4][CW], k[4][CW], a[4][CW], d[16];
#pragma unroll
      for (int t = 0; t < 4; t++) {
        gl_ld_bf16<CW>(rq + t * DP, q[t]);
        gl_ld_bf16<CW>(rk + t * DP, k[t]);
        gl_ld_f32<CW>(rz + t * DP, a[t]);
#pragma unroll
        for (int i = 0; i < CW; i++) {
          q[t][i] *= scale;
          a[t][i] = blk * 4 + t < n ? gl_decay(a[t][i], inv_tau) : 1.0f;
        }
      }
#pragma unroll
      for (int i = 0; i < 16; i++) d[i] = 0.0f;
#pragma unroll
      for (int t = 0; t < 4; t++)
#pragma unroll
        for (int i = 0; i < CW; i++) {
          float x = q[t][i];
#pragma unroll
          for (int u = t; u >= 0; u--) {
            d[t * 4 + u] = fmaf(x, k[u][i], d[t * 4 + u]);
            x *= a[u][i];
          }
          q[t][i] = x;  // times the decays from the block's first token to t
        }
      float f[CW];
#pragma unroll
      for (int i = 0; i < CW; i++) f[i] = 1.0f;
#pragma unroll
      for (int t = 3; t >= 0; t--)
#pragma unroll
        for (int i = 0; i < CW; i++) {
          k[t][i] *= f[i];
          f[i] *= a[t][i];
        }
#pragma unroll
      for (int t = 0; t < 4; t++) {
        gl_st_f32<CW>(s_q + (blk * 4 + t) * DP + c, q[t]);
        gl_st_f32<CW>(s_k + (blk * 4 + t) * DP + c, k[t]);
      }
      gl_st_f32<CW>(s_a + blk * DP + c, f);
      // sums over the warp, every step leaving a lane half of its values
#pragma unroll
      for (int x = 16, m = 8; m > 0; x >>= 1, m >>= 1) {
        const bool up = (lane & x) != 0;
#pragma unroll
        for (int i = 0; i < 8; i++)
          if (i < m) {
            const float mine = up ? d[i + m] : d[i], other = up ? d[i] : d[i + m];
            d[i] = mine + __shfl_xor_sync(0xffffffffu, other, x);
          }
      }
      d[0] += __shfl_xor_sync(0xffffffffu, d[0], 1);
      if (!(lane & 1)) s_d[blk * 16 + (lane >> 1)] = d[0];
    }
    gl_sync<C::THREADS>();
#pragma unroll 1
    for (int blk = 0; blk < C::NB; blk++) {
      float o[4 * CPT];
#pragma unroll
      for (int t = 0; t < 4; t++) {
        const float4* pq = reinterpret_cast<const float4*>(s_q + (blk * 4 + t) * DP) + l;
        float2 oa[CPT];
#pragma unroll
        for (int c = 0; c < CPT; c++) oa[c] = make_float2(0.0f, 0.0f);
#pragma unroll
        for (int i = 0; i < KV; i++) {
          const float4 q = pq[i * LPC];
#pragma unroll
          for (int c = 0; c < CPT; c++) {
            oa[c] = gl_fma2(make_float2(q.x, q.y), s[c][2 * i], oa[c]);
            oa[c] = gl_fma2(make_float2(q.z, q.w), s[c][2 * i + 1], oa[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < CPT; c++) o[t * CPT + c] = oa[c].x + oa[c].y;
      }
      {
        const float4* pa = reinterpret_cast<const float4*>(s_a + blk * DP) + l;
#pragma unroll
        for (int i = 0; i < KV; i++) {
          const float4 a = pa[i * LPC];
#pragma unroll
          for (int c = 0; c < CPT; c++) {
            s[c][2 * i] = gl_mul2(make_float2(a.x, a.y), s[c][2 * i]);
            s[c][2 * i + 1] = gl_mul2(make_float2(a.z, a.w), s[c][2 * i + 1]);
          }
        }
      }
#pragma unroll
      for (int t = 0; t < 4; t++) {
        const float4* pk = reinterpret_cast<const float4*>(s_k + (blk * 4 + t) * DP) + l;
        float v[CPT];
        gl_ld_bf16<CPT>(rv + (blk * 4 + t) * EC + c0, v);
        float4 k[KV];
#pragma unroll
        for (int i = 0; i < KV; i++) k[i] = pk[i * LPC];
#pragma unroll
        for (int c = 0; c < CPT; c++) {
          const float2 vv = make_float2(v[c], v[c]);
#pragma unroll
          for (int i = 0; i < KV; i++) {
            s[c][2 * i] = gl_fma2(make_float2(k[i].x, k[i].y), vv, s[c][2 * i]);
            s[c][2 * i + 1] = gl_fma2(make_float2(k[i].z, k[i].w), vv, s[c][2 * i + 1]);
          }
        }
      }
      // sums over a column's lanes, halving: lane l ends with values l * M .. l * M + M - 1 of [token][column]
#pragma unroll
      for (int x = LPC / 2, m = 2 * CPT; x > 0; x >>= 1, m >>= 1) {
        const bool up = (l & x) != 0;
#pragma unroll
        for (int i = 0; i < 2 * CPT; i++)
          if (i < m) {
            const float mine = up ? o[i + m] : o[i], other = up ? o[i] : o[i + m];
            o[i] = mine + __shfl_xor_sync(0xffffffffu, other, x);
          }
      }
      const int t = l * M / CPT, c = l * M % CPT;
      const float4 d = *reinterpret_cast<const float4*>(s_d + blk * 16 + t * 4);  // zero for later tokens
      const float dd[4] = {d.x, d.y, d.z, d.w};
      float r[M];
#pragma unroll
      for (int i = 0; i < M; i++) r[i] = o[i];
#pragma unroll
      for (int u = 0; u < 4; u++) {
        float w[M];
        gl_ld_bf16<M>(rv + (blk * 4 + u) * EC + c0 + c, w);
#pragma unroll
        for (int i = 0; i < M; i++) r[i] = fmaf(dd[u], w[i], r[i]);
      }
      if (WHOLE) gl_st_f32<M>(s_o + (blk * 4 + t) * EC + c0 + c, r);
      else if (blk * 4 + t < n && c0 + c < cols) gl_st_f32<M>(p.raw + ((row0 + t0 + blk * 4 + t) * p.heads + head) * vdim + e0 + c0 + c, r);
    }
    if (WHOLE) {
      gl_sync<C::THREADS>();
      // output norm and gate: a warp per token
      const uint16_t* rg = reinterpret_cast<const uint16_t*>(rw + C::RG);
      const int c = lane * C::OW;
      uint16_t* out = reinterpret_cast<uint16_t*>(p.out) + (row0 + t0) * p.ldo + head * vdim + c;
      for (int t = warp; t < n; t += C::NW) {
        float x[C::OW], g[C::OW], ss = 0.0f;
        gl_ld_f32<C::OW>(s_o + t * EC + c, x);
        gl_ld_bf16<C::OW>(rg + t * EC + c, g);
#pragma unroll
        for (int i = 0; i < C::OW; i++) ss = fmaf(x[i], x[i], ss);
        if (c >= cols) ss = 0.0f;
        const float rms = rsqrtf(hy_warp_sum(ss) / (float)vdim + p.eps);
#pragma unroll
        for (int i = 0; i < C::OW; i++) x[i] = x[i] * rms * nw[i] * gl_silu(g[i]);
        if (c < cols) {
          uint16_t* dst = out + (int64_t)t * p.ldo;
          if constexpr (C::OW == 1) {
            dst[0] = f32_to_bf16_bits(x[0]);
          } else {
#pragma unroll
            for (int i = 0; i < C::OW; i += 2) {
              const __nv_bfloat162 w = __floats2bfloat162_rn(x[i], x[i + 1]);
              *reinterpret_cast<__nv_bfloat162*>(dst + i) = w;
            }
          }
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < KP; i++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int k = (i >> 1) * 4 * LPC + l * 4 + (i & 1) * 2 + e;
#pragma unroll
      for (int c = 0; c < CPT; c += 4)
        if (k < dim && c0 + c < cols)
          *reinterpret_cast<float4*>(st + (int64_t)k * vdim + c) =
              e ? make_float4(s[c][i].y, s[c + 1][i].y, s[c + 2][i].y, s[c + 3][i].y) : make_float4(s[c][i].x, s[c + 1][i].x, s[c + 2][i].x, s[c + 3][i].x);
    }
}

static int gla_opt_in(const void* k, size_t smem, bool (&opted)[16]) {
  int dev = 0;
  cudaGetDevice(&dev);
  if (smem > 48 * 1024 && (dev < 0 || dev >= 16 || !opted[dev])) {
    TPX_CUDA_OK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  return TPX_OK;
}

static int gla_out(const TpxGla& p, cudaStream_t st) {
  void (*k)(TpxGla) = p.f32 ? gla_out_kernel<float> : gla_out_kernel<__nv_bfloat16>;
  TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)((p.B * p.S * p.heads + 7) / 8)), dim3(256), 0, st, p));
  return TPX_OK;
}

template <int DP, int EC, int LPC, int CPT, int TC, bool WHOLE>
static int gla_fast_launch(const TpxGla& p, cudaStream_t st) {
  using C = GfCfg<DP, EC, LPC, CPT, TC, WHOLE>;
  static bool opted[16] = {};
  void (*k)(TpxGla) = gla_fast_kernel<DP, EC, LPC, CPT, TC, WHOLE>;
  const int rc = gla_opt_in((const void*)k, C::SMEM, opted);
  if (rc) return rc;
  TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)p.heads, (unsigned)(WHOLE ? 1 : (p.vdim + EC - 1) / EC), (unsigned)p.B), dim3(C::THREADS), C::SMEM, st, p));
  return WHOLE ? TPX_OK : gla_out(p, st);
}

static bool gla_fast_serves(const TpxGla& a) {
  return !a.f32 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.ldp % 8 == 0 && a.q_col % 8 == 0 && a.k_col % 8 == 0 && a.v_col % 8 == 0 &&
         a.g_col % 8 == 0 && a.ldp < (1ll << 30) && a.heads * a.dim < (1ll << 30) &&
         a.ldo % 8 == 0 && (((uintptr_t)a.proj | (uintptr_t)a.zraw | (uintptr_t)a.state | (uintptr_t)a.raw | (uintptr_t)a.out) & 15) == 0;
}

static int gla_fast(const TpxGla& a, cudaStream_t st) {
  // whole heads per CTA when there are many, columns cut over CTAs when a token's latency counts
  const bool many = a.vdim <= 256 && a.B * a.heads >= 2 * sm_count();
  if (a.dim <= 32) {
    if (!many) return gla_fast_launch<32, 32, 8, 4, 16, false>(a, st);
    return a.vdim <= 64 ? gla_fast_launch<32, 64, 4, 8, 8, true>(a, st) : a.vdim <= 128 ? gla_fast_launch<32, 128, 4, 8, 8, true>(a, st)
                                                                                       : gla_fast_launch<32, 256, 4, 8, 8, true>(a, st);
  }
  if (a.dim <= 64) {
    if (!many) return gla_fast_launch<64, 32, 16, 4, 16, false>(a, st);
    return a.vdim <= 64 ? gla_fast_launch<64, 64, 4, 8, 16, true>(a, st) : a.vdim <= 128 ? gla_fast_launch<64, 128, 4, 8, 16, true>(a, st)
                                                                                       : gla_fast_launch<64, 256, 4, 8, 16, true>(a, st);
  }
  if (!many) return gla_fast_launch<128, 32, 16, 4, 16, false>(a, st);
  return a.vdim <= 64 ? gla_fast_launch<128, 64, 8, 8, 8, true>(a, st) : a.vdim <= 128 ? gla_fast_launch<128, 128, 8, 8, 8, true>(a, st)
                                                                                      : gla_fast_launch<128, 256, 8, 8, 8, true>(a, st);
}

template <typename T, int DP>
static int gla_launch(const TpxGla& p, cudaStream_t st) {
  using C = GlaCfg<DP>;
  static bool opted[16] = {};
  const int rc = gla_opt_in((const void*)gla_kernel<T, DP>, C::SMEM, opted);
  if (rc) return rc;
  TPX_CUDA_OK(launch_pdl(gla_kernel<T, DP>, dim3((unsigned)p.heads, (unsigned)((p.vdim + C::COLS - 1) / C::COLS), (unsigned)p.B), dim3(128), C::SMEM, st, p));
  return gla_out(p, st);
}

template <typename T>
static int gla_run(const TpxGla& a, cudaStream_t st) {
  if (a.dim <= 16) return gla_launch<T, 16>(a, st);
  if (a.dim <= 32) return gla_launch<T, 32>(a, st);
  if (a.dim <= 64) return gla_launch<T, 64>(a, st);
  if (a.dim <= 128) return gla_launch<T, 128>(a, st);
  if (a.dim <= 256) return gla_launch<T, 256>(a, st);
  return gla_launch<T, 512>(a, st);
}

static int gla_token(const TpxGla& a, cudaStream_t st) {
  const int64_t ncg = a.vdim / 4, nrg = kGlaTokThreads / ncg, d3 = 3 * a.dim;
  const size_t smem = (size_t)((d3 + 3) / 4 * 4 + nrg * ncg * 4) * 4;
  void (*k)(TpxGla) = a.f32 ? gla_token_kernel<float> : gla_token_kernel<__nv_bfloat16>;
  TPX_CUDA_OK(launch_pdl(k, dim3((unsigned)a.heads, (unsigned)a.B), dim3(kGlaTokThreads), smem, st, a));
  return TPX_OK;
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_gla_token_serves(int64_t dim, int64_t vdim) { return dim > 0 && dim <= 512 && vdim > 0 && vdim % 4 == 0 && vdim <= 4 * kGlaTokThreads; }

extern "C" int tpx_gla(const TpxGla* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "gla: null argument block");
  TPX_REQUIRE(a->B >= 0 && a->S >= 0 && a->heads > 0 && a->dim > 0 && a->vdim > 0 && a->past >= 0 && a->tau > 0.0f, TPX_ERR_ARG, "gla: bad shape");
  TPX_REQUIRE(a->dim <= 512, TPX_ERR_UNSUPPORTED, "gla: heads of at most 512 key channels, got %ld", (long)a->dim);
  TPX_REQUIRE(a->B <= 65535 && a->S < (1 << 24) && a->past < (1ll << 30) && a->heads < (1 << 16) && a->vdim < (1 << 20), TPX_ERR_ARG, "gla: shape too large");
  if (a->B == 0 || a->S == 0) return TPX_OK;
  TPX_REQUIRE(a->proj && a->norm_w && a->state && a->out, TPX_ERR_ARG, "gla: null pointer");
  const int64_t hd = a->heads * a->dim, he = a->heads * a->vdim;
  TPX_REQUIRE(a->q_col >= 0 && a->k_col >= 0 && a->v_col >= 0 && a->g_col >= 0 && a->q_col + hd <= a->ldp && a->k_col + hd <= a->ldp && a->v_col + he <= a->ldp &&
                  a->g_col + he <= a->ldp && a->ldo >= he, TPX_ERR_ARG, "gla: columns outside their rows");
  TPX_REQUIRE(!a->dev_len || a->S == 1, TPX_ERR_ARG, "gla: dev_len is for single tokens");
  const bool token = a->S == 1 && tpx_gla_token_serves(a->dim, a->vdim) && ((uintptr_t)a->state & 15) == 0;
  TPX_REQUIRE(a->zraw || (token && a->a2 && a->a2_bias && a->rank > 0 && a->lda2 >= a->rank && a->a1_col >= 0 && a->a1_col + a->rank <= a->ldp), TPX_ERR_ARG,
              "gla: the decay's input is missing");
  cudaStream_t st = (cudaStream_t)stream;
  if (token) return gla_token(*a, st);
  TPX_REQUIRE(a->raw, TPX_ERR_ARG, "gla: null pointer");
  if (gla_fast_serves(*a)) return gla_fast(*a, st);
  return a->f32 ? gla_run<float>(*a, st) : gla_run<__nv_bfloat16>(*a, st);
}
