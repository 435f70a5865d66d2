// Decoding with latent attention in bf16: the per-head maps (keys into the query, latents into values) as small grouped
// matrix products, and attention of all heads over the cached latents, each read once.
//
// Attention: a thread-block cluster per (sequence, group of 32 heads); its CTAs share the window's keys in tiles of 32.
// A tile is a page's 32 rows of one sequence, contiguous in the cache: one bulk copy, four of them in flight (a copy per
// row, or cp.async, spent a quarter of the kernel's time on requests). The cache rows carry 8 elements of padding so that
// rows lie in different banks as they are. Rows of a page outside the window are cleared after the copy. Eight warps: each computes
// the part of the scores of 16 keys and all heads that a quarter of the row contributes (its slice of the queries stays in
// registers: read from shared memory by every warp it would be the largest traffic there), the softmax of 4 heads, and the
// weighted sum of its eighth of the latent columns for all heads (mma.sync bf16, fp32 accumulation; a latent row is key
// and value at once). The scores of a tile are computed beside the weighted sum of the tile before it: two barriers per
// tile, and independent MMAs between them. The weights are multiplied as two bf16 terms, so that they keep their 32-bit
// value in effect. The CTAs of a cluster merge through distributed shared memory: nothing partial goes to global memory.
#include "tpx_hybrid.cuh"
#include "tpx_tc_ptx.cuh"

namespace tpx {

__device__ __forceinline__ void ld_cp16(uint32_t dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void ld_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ld_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldm_x4(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldm_x4t(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldm_x2(uint32_t a, uint32_t (&r)[2]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldm_x2t(uint32_t a, uint32_t (&r)[2]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a) : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t ld_pack(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// ---------------------------------------------------------------- grouped products
struct GroupedParams {
  const uint16_t *w, *x;
  uint16_t* out;
  const float* gate;                // value map: [T][groups]
  long long ldx, xg, ldo, og, ldw;  // strides: x token, x group, out token, out group, w row
  int T, N, K, KP;                  // KP: K rounded up to 16
  int groups;
  // key map: the rotated query part
  const float* cos_sin;
  int dim, rot, krp, R;
  long long pad0, pad1;             // value map: columns [pad0, pad1) of an output row are set to zero
};

// TRANS: w[group][k][n] (rows of one k), else w[group][n][k]. 4 warps x NT8 tiles of 8 outputs; 16 tokens at a time.
template <int NT8, bool TRANS>
__global__ void __launch_bounds__(128) grouped_mma_kernel(GroupedParams p) {
  constexpr int NT = 32 * NT8;
  extern __shared__ __align__(16) unsigned char gr_smem[];
  const int g = blockIdx.x, n0 = blockIdx.y * NT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ldws = TRANS ? NT + 8 : p.KP + 8, ldxs = p.KP + 8;
  uint16_t* sw = reinterpret_cast<uint16_t*>(gr_smem);
  uint16_t* sx = sw + (size_t)(TRANS ? p.KP : NT) * ldws;
  pdl_trigger();
  if (TRANS && n0 >= p.N) {  // the last block of a group: the rotated part of the queries
    pdl_wait();
    const int rw = p.R - p.krp, half = p.rot / 2;
    for (int i = threadIdx.x; i < p.T * rw; i += 128) {
      const int j = i / rw, e = i % rw;
      float v = 0.0f;
      if (e < p.rot) {
        const float2 r = reinterpret_cast<const float2*>(p.cos_sin)[(int64_t)j * half + (e >> 1)];
        const uint16_t* qr = p.x + j * p.ldx + g * p.xg + p.dim;
        const float a = bf16_bits_to_f32(qr[e & ~1]), b = bf16_bits_to_f32(qr[e | 1]);
        v = (e & 1) ? b * r.x + a * r.y : a * r.x - b * r.y;
      }
      p.out[j * p.ldo + g * p.og + p.krp + e] = f32_to_bf16_bits(v);
    }
    return;
  }
  // weights do not depend on earlier kernels
  if (TRANS) {
    for (int i = threadIdx.x; i < p.KP * (NT / 8); i += 128) {
      const int r = i / (NT / 8), c = (i % (NT / 8)) * 8;
      const bool ok = r < p.K && n0 + c < p.N;
      ld_cp16(tc_smem_u32(sw + r * ldws + c), ok ? p.w + ((long long)g * p.K + r) * p.ldw + n0 + c : p.w, ok);
    }
  } else {
    const int kc = p.KP / 8;
    for (int i = threadIdx.x; i < NT * kc; i += 128) {
      const int r = i / kc, c = (i % kc) * 8;
      const bool ok = n0 + r < p.N;
      ld_cp16(tc_smem_u32(sw + r * ldws + c), ok ? p.w + ((long long)g * p.N + n0 + r) * p.ldw + c : p.w, ok);
    }
  }
  ld_commit();
  pdl_wait();
  const int kc = p.KP / 8;
  for (int t0 = 0; t0 < p.T; t0 += 16) {
    if (t0) __syncthreads();
    for (int i = threadIdx.x; i < 16 * kc; i += 128) {
      const int r = i / kc, c = (i % kc) * 8;
      const bool ok = t0 + r < p.T && c < p.K;
      ld_cp16(tc_smem_u32(sx + r * ldxs + c), ok ? p.x + (t0 + r) * p.ldx + g * p.xg + c : p.x, ok);
    }
    ld_commit();
    ld_wait<0>();
    __syncthreads();
    float acc[NT8][4] = {};
    const uint32_t xa = tc_smem_u32(sx + (lane & 15) * ldxs + (lane >> 4) * 8);
    for (int k = 0; k < p.KP; k += 16) {
      uint32_t a[4];
      ldm_x4(xa + k * 2, a);
#pragma unroll
      for (int i = 0; i < NT8; i++) {
        const int n = (warp * NT8 + i) * 8;
        uint32_t b[2];
        if (TRANS) ldm_x2t(tc_smem_u32(sw + (k + (lane & 15)) * ldws + n), b);
        else ldm_x2(tc_smem_u32(sw + (n + (lane & 7)) * ldws + k + ((lane >> 3) & 1) * 8), b);
        mma16816(acc[i], a, b[0], b[1]);
      }
    }
#pragma unroll
    for (int h = 0; h < 2; h++) {
      const int t = t0 + (lane >> 2) + h * 8;
      if (t < p.T) {
        const float s = p.gate ? p.gate[(long long)t * p.groups + g] : 1.0f;
#pragma unroll
        for (int i = 0; i < NT8; i++) {
          const int n = n0 + (warp * NT8 + i) * 8 + (lane & 3) * 2;
          uint16_t* o = p.out + t * p.ldo + g * p.og + n;
          if (n < p.N) o[0] = f32_to_bf16_bits(acc[i][2 * h] * s);
          if (n + 1 < p.N) o[1] = f32_to_bf16_bits(acc[i][2 * h + 1] * s);
        }
      }
    }
  }
  if (!TRANS && g == 0 && blockIdx.y == 0)
    for (int t = 0; t < p.T; t++)
      for (long long c = p.pad0 + threadIdx.x; c < p.pad1; c += 128) p.out[t * p.ldo + c] = 0;
}

template <int NT8, bool TRANS>
static int grouped_launch(const GroupedParams& p, int extra_blocks, cudaStream_t st) {
  constexpr int NT = 32 * NT8;
  const size_t smem = ((size_t)(TRANS ? p.KP : NT) * (TRANS ? NT + 8 : p.KP + 8) + (size_t)16 * (p.KP + 8)) * 2;
  TPX_REQUIRE(smem <= 220 * 1024, TPX_ERR_UNSUPPORTED, "latent decode: per-head map too large (contraction of %d)", p.K);
  static bool opted[16] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 16 || !opted[dev]) {
    TPX_CUDA_OK(cudaFuncSetAttribute(grouped_mma_kernel<NT8, TRANS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  TPX_CUDA_OK(launch_pdl(grouped_mma_kernel<NT8, TRANS>, dim3((unsigned)p.groups, (unsigned)((p.N + NT - 1) / NT + extra_blocks)), dim3(128), smem, st, p));
  return TPX_OK;
}

bool latent_absorb_mma_serves(const TpxLatentAbsorb& a) {
  return !a.f32 && a.T <= 64 && a.dim % 8 == 0 && (a.dim + a.rot_dim) % 8 == 0 && a.ldq % 8 == 0 && a.krp % 8 == 0 && a.dim <= 512 &&
         (((uintptr_t)a.q | (uintptr_t)a.w_uk) & 15) == 0;
}
int latent_absorb_mma(const TpxLatentAbsorb& a, cudaStream_t st) {
  GroupedParams p = {};
  p.w = (const uint16_t*)a.w_uk; p.x = (const uint16_t*)a.q; p.out = (uint16_t*)a.qa;
  p.ldx = a.ldq; p.xg = a.dim + a.rot_dim; p.ldo = a.heads * a.R; p.og = a.R; p.ldw = a.krp;
  p.T = (int)a.T; p.N = (int)a.krp; p.K = (int)a.dim; p.KP = (int)((a.dim + 15) / 16 * 16); p.groups = (int)a.heads;
  p.cos_sin = a.cos_sin; p.dim = (int)a.dim; p.rot = (int)a.rot_dim; p.krp = (int)a.krp; p.R = (int)a.R;
  return grouped_launch<2, true>(p, a.R > a.krp ? 1 : 0, st);
}
bool latent_value_mma_serves(const TpxLatentValue& a) {
  return !a.f32 && a.T <= 64 && a.krp % 16 == 0 && a.krp <= 1152 && (((uintptr_t)a.ol | (uintptr_t)a.w_uv) & 15) == 0;
}
int latent_value_mma(const TpxLatentValue& a, cudaStream_t st) {
  GroupedParams p = {};
  p.w = (const uint16_t*)a.w_uv; p.x = (const uint16_t*)a.ol; p.out = (uint16_t*)a.out; p.gate = a.gate;
  p.ldx = a.heads * a.krp; p.xg = a.krp; p.ldo = a.ldo; p.og = a.vdim; p.ldw = a.krp;
  p.T = (int)a.T; p.N = (int)a.vdim; p.K = (int)a.krp; p.KP = (int)a.krp; p.groups = (int)a.heads;
  p.pad0 = a.heads * a.vdim; p.pad1 = a.ldo;
  return grouped_launch<1, false>(p, 0, st);
}

// ---------------------------------------------------------------- attention
static __device__ unsigned g_latent_dec_err;  // set when a bounded wait gave up; read and cleared by tpx_latent_decode_status
constexpr int kLdKeys = 32, kLdStages = 4, kLdWarps = 8, kLdThreads = 256;

// MT: 16-head tiles per CTA; CW: 8-column latent tiles per warp (krp <= CW * 64); KS: 16-value steps of a quarter row
template <int MT, int CW, int KS>
__global__ void __launch_bounds__(kLdThreads, 1) latent_decode_kernel(TpxLatentAttn p, int splits) {
  constexpr int MR = MT * 16, SW = kLdKeys + 4, PW = kLdKeys + 8;
  extern __shared__ __align__(16) unsigned char ld_smem[];
  const int R = (int)p.R, krp = (int)p.krp, lds = R;
  uint16_t* sk = reinterpret_cast<uint16_t*>(ld_smem);                 // [stages][32][R]
  uint16_t* sp = sk + (size_t)kLdStages * kLdKeys * lds;               // [2 terms][MR][32 + 8]
  float* ss = reinterpret_cast<float*>(sp + 2 * MR * (kLdKeys + 8));   // [4 quarters][MR][32 + 4]
  float* sm = ss + 4 * MR * SW;                                        // [MR] running maxima (log2 units)
  float* sl = sm + MR;                                                 // [MR] running sums
  float* sa = sl + MR;                                                 // [MR] rescaling of this tile
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rank = blockIdx.x % splits, b = blockIdx.x / splits, h0 = blockIdx.y * MR;
  const int kq = warp & 3, key0 = (warp >> 2) * 16;
  __shared__ __align__(8) unsigned long long full[kLdStages];
  pdl_trigger();
  if (threadIdx.x == 0) {
    for (int i = 0; i < kLdStages; i++) tc_mbar_init(tc_smem_u32(&full[i]), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  __syncthreads();
  pdl_wait();
  const int64_t t = p.dev_len ? *p.dev_len : p.past;
  const int64_t lo = max((int64_t)(p.start ? p.start[b] : 0), t - p.window + 1);
  const int blk0 = (int)(lo / kLdKeys), tiles = (int)(t / kLdKeys) - blk0 + 1;  // tile i: the keys of page blk0 + i
  const int i0 = (int)((long long)tiles * rank / splits), i1 = (int)((long long)tiles * (rank + 1) / splits);
  const int np = (int)p.npages;
  auto fetch = [&](int i) {  // one thread
    const uint32_t bar = tc_smem_u32(&full[(i - i0) % kLdStages]);
    const uint16_t* src = reinterpret_cast<const uint16_t*>(__ldg(p.pages + (blk0 + i) % np)) + (int64_t)b * kLdKeys * R;
    tc_mbar_expect_tx(bar, (uint32_t)(kLdKeys * R * 2));
    tc_bulk_g2s(tc_smem_u32(sk + (size_t)((i - i0) % kLdStages) * kLdKeys * lds), src, (uint32_t)(kLdKeys * R * 2), bar);
  };
  bool dead = false;
  auto arrived = [&](int i) {  // tile i is in shared memory
    if (!dead && !tc_wait(tc_smem_u32(&full[(i - i0) % kLdStages]), (uint32_t)(((i - i0) / kLdStages) & 1))) {
      dead = true;
      atomicExch(&g_latent_dec_err, 1u);
    }
    const int64_t k0 = (int64_t)(blk0 + i) * kLdKeys;
    if (k0 < lo || k0 + kLdKeys - 1 > t) {  // the first and the last page: what lies outside may be anything
      uint16_t* kt = sk + (size_t)((i - i0) % kLdStages) * kLdKeys * lds;
      for (int q = threadIdx.x; q < kLdKeys * (R / 8); q += kLdThreads) {
        const int64_t key = k0 + q / (R / 8);
        if (key < lo || key > t) *reinterpret_cast<uint4*>(kt + q * 8) = make_uint4(0, 0, 0, 0);
      }
      __syncthreads();
    }
  };
  if (threadIdx.x == 0)
    for (int i = i0; i < min(i1, i0 + kLdStages - 1); i++) fetch(i);
  // this warp's quarter of the queries as MMA operands
  const int ksteps = (R - 8) / 16, k0 = kq * ((ksteps + 3) / 4), k1 = min(ksteps, k0 + (ksteps + 3) / 4);
  uint32_t qf[MT][KS][4];
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int k = 0; k < KS; k++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int h = h0 + m * 16 + (lane >> 2) + (e & 1) * 8, c = (k0 + k) * 16 + (e >> 1) * 8 + (lane & 3) * 2;
        qf[m][k][e] = (k0 + k < k1 && h < p.heads)
                          ? __ldg(reinterpret_cast<const uint32_t*>(reinterpret_cast<const uint16_t*>(p.qa) + ((int64_t)b * p.heads + h) * R + c)) : 0u;
      }
  for (int i = threadIdx.x; i < MR; i += kLdThreads) { sm[i] = -INFINITY; sl[i] = 0.0f; }
  float o[MT][CW][4];
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int c = 0; c < CW; c++)
#pragma unroll
      for (int e = 0; e < 4; e++) o[m][c][e] = 0.0f;
  const float sc2 = p.scale * 1.4426950408889634f;
  const int cols = (krp / 16 + kLdWarps - 1) / kLdWarps * 2;  // 8-column tiles per warp, in pairs
  const int ct0 = warp * cols;
  // No branch inside the MMA loops, so that their loads run ahead: steps and tiles this warp does not have read some other
  // valid place, against zero queries or into accumulators that are dropped
  // scores of the warp's 16 keys and quarter row, from stage st
  auto scores = [&](int st, float (&acc)[MT][2][4]) {
    const uint32_t kb = tc_smem_u32(sk + ((size_t)st * kLdKeys + key0 + (lane & 7) + ((lane >> 4) & 1) * 8) * lds + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int k = 0; k < KS; k++) {
      uint32_t b[4];
      ldm_x4(kb + min(k0 + k, ksteps - 1) * 32, b);
#pragma unroll
      for (int m = 0; m < MT; m++) {
        mma16816(acc[m][0], qf[m][k], b[0], b[1]);
        mma16816(acc[m][1], qf[m][k], b[2], b[3]);
      }
    }
  };
  auto put_scores = [&](const float (&acc)[MT][2][4]) {
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int n = 0; n < 2; n++)
#pragma unroll
        for (int h = 0; h < 2; h++)
          *reinterpret_cast<float2*>(ss + (kq * MR + m * 16 + (lane >> 2) + h * 8) * SW + key0 + n * 8 + (lane & 3) * 2) =
              make_float2(acc[m][n][2 * h], acc[m][n][2 * h + 1]);
  };
  // softmax of this warp's MR / 8 heads, all at once: LR lanes per head, KL neighbouring keys per lane
  auto softmax = [&](int i) {
    constexpr int LR = 32 / (MR / kLdWarps), KL = kLdKeys / LR;
    const int64_t key0 = (int64_t)(blk0 + i) * kLdKeys;
    const int from = (int)max((int64_t)0, lo - key0), left = (int)min((int64_t)kLdKeys, t - key0 + 1);  // keys from .. left - 1 count
    const int r = warp * (MR / kLdWarps) + lane / LR, k = (lane % LR) * KL;
    float x[KL] = {};
#pragma unroll
    for (int q = 0; q < 4; q++)
#pragma unroll
      for (int e = 0; e < KL; e += 2) {
        const float2 u = *reinterpret_cast<const float2*>(ss + (q * MR + r) * SW + k + e);
        x[e] += u.x;
        x[e + 1] += u.y;
      }
    float mx = -INFINITY;
#pragma unroll
    for (int e = 0; e < KL; e++) {
      x[e] = k + e >= from && k + e < left ? x[e] * sc2 : -INFINITY;
      mx = fmaxf(mx, x[e]);
    }
#pragma unroll
    for (int d = LR / 2; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
    const float mo = sm[r], mn = fmaxf(mo, mx);  // a tile has at least one key
    float sum = 0.0f;
    uint16_t* ph = sp + r * PW + k;
#pragma unroll
    for (int e = 0; e < KL; e += 2) {
      const float e0 = exp2f(x[e] - mn), e1 = exp2f(x[e + 1] - mn);
      sum += e0 + e1;
      const uint32_t hi = ld_pack(e0, e1);
      *reinterpret_cast<uint32_t*>(ph + e) = hi;
      *reinterpret_cast<uint32_t*>(ph + MR * PW + e) = ld_pack(e0 - __uint_as_float(hi << 16), e1 - __uint_as_float(hi & 0xffff0000u));
    }
#pragma unroll
    for (int d = LR / 2; d > 0; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
    __syncwarp();
    if (lane % LR == 0) {
      const float al = exp2f(mo - mn);
      sm[r] = mn;
      sl[r] = sl[r] * al + sum;
      sa[r] = al;
    }
  };
  if (i0 < i1) {
    arrived(i0);
    float acc[MT][2][4] = {};
    scores(0, acc);
    put_scores(acc);
  }
  __syncthreads();
  if (i0 < i1) softmax(i0);
  // one round: the scores of tile i + 1 beside the weighted sum of tile i, then the softmax of tile i + 1
  for (int i = i0; i < i1; i++) {
    const int st = (i - i0) % kLdStages;
    __syncthreads();  // the weights of tile i are there, tile i - 1 is no longer read
    if (threadIdx.x == 0 && i + kLdStages - 1 < i1) fetch(i + kLdStages - 1);
    if (i + 1 < i1) arrived(i + 1);
    float acc[MT][2][4] = {};
    scores((st + 1) % kLdStages, acc);  // behind the last tile: of whatever is there, not used
    bool scale = false;
#pragma unroll
    for (int m = 0; m < MT; m++) scale |= sa[m * 16 + (lane >> 2)] != 1.0f || sa[m * 16 + (lane >> 2) + 8] != 1.0f;
    if (__any_sync(0xffffffffu, scale)) {
#pragma unroll
      for (int m = 0; m < MT; m++) {
        const float a0 = sa[m * 16 + (lane >> 2)], a1 = sa[m * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int c = 0; c < CW; c++) { o[m][c][0] *= a0; o[m][c][1] *= a0; o[m][c][2] *= a1; o[m][c][3] *= a1; }
      }
    }
    const uint16_t* kt = sk + (size_t)st * kLdKeys * lds;
#pragma unroll
    for (int k = 0; k < kLdKeys; k += 16) {
      uint32_t a[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; m++)
#pragma unroll
        for (int term = 0; term < 2; term++) ldm_x4(tc_smem_u32(sp + (term * MR + m * 16 + (lane & 15)) * PW + k + (lane >> 4) * 8), a[m][term]);
#pragma unroll
      for (int c = 0; c < CW; c += 2) {
        const int n = min((ct0 + c) * 8, krp - 16);
        uint32_t bb[4];
        ldm_x4t(tc_smem_u32(kt + (k + (lane & 15)) * lds + n + (lane >> 4) * 8), bb);
#pragma unroll
        for (int term = 0; term < 2; term++)
#pragma unroll
          for (int m = 0; m < MT; m++) {
            mma16816(o[m][c], a[m][term], bb[0], bb[1]);
            mma16816(o[m][c + 1], a[m][term], bb[2], bb[3]);
          }
      }
    }
    put_scores(acc);
    __syncthreads();
    if (i + 1 < i1) softmax(i + 1);
  }
  // merge: every CTA scales its sums to the cluster's maximum and total, then adds up its share of the columns
  __syncthreads();
  tc_cluster_sync();
  float* so = reinterpret_cast<float*>(ld_smem);  // [MR][krp], over the key stages
  if (threadIdx.x < MR * 8) {  // eight lanes per head, one per CTA of the cluster
    const int r = threadIdx.x >> 3, c = threadIdx.x & 7;
    float m = -INFINITY, l = 0.0f;
    if (c < splits) {
      asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(m) : "r"(tc_mapa(tc_smem_u32(sm + r), c)) : "memory");
      asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(l) : "r"(tc_mapa(tc_smem_u32(sl + r), c)) : "memory");
    }
    float mx = m;
#pragma unroll
    for (int x = 4; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
    float tot = l > 0.0f ? l * exp2f(m - mx) : 0.0f;
#pragma unroll
    for (int x = 4; x > 0; x >>= 1) tot += __shfl_xor_sync(0xffffffffu, tot, x);
    if (c == 0) sa[r] = sl[r] > 0.0f ? exp2f(sm[r] - mx) / tot : 0.0f;
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; m++) {
    const int r = m * 16 + (lane >> 2);
    const float a0 = sa[r], a1 = sa[r + 8];
#pragma unroll
    for (int c = 0; c < CW; c++) {
      const int n = (ct0 + c) * 8 + (lane & 3) * 2;
      if (c < cols && n < krp) {
        *reinterpret_cast<float2*>(so + r * krp + n) = make_float2(o[m][c][0] * a0, o[m][c][1] * a0);
        *reinterpret_cast<float2*>(so + (r + 8) * krp + n) = make_float2(o[m][c][2] * a1, o[m][c][3] * a1);
      }
    }
  }
  tc_cluster_sync();
  const int nq = MR * krp / 4;
  for (int q = rank * kLdThreads + threadIdx.x; q < nq; q += splits * kLdThreads) {
    float s[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    tc_cluster_sum<1, 8>(tc_smem_u32(so + q * 4), splits, s);
    const int r = q * 4 / krp, n = q * 4 % krp;
    if (h0 + r < p.heads)
      *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(p.ol) + ((int64_t)b * p.heads + h0 + r) * krp + n) = make_uint2(ld_pack(s[0], s[1]), ld_pack(s[2], s[3]));
  }
  tc_cluster_sync();  // nobody leaves while its shared memory is being read
}

static size_t ld_smem_bytes(int MR, int R) {
  return ((size_t)kLdStages * kLdKeys * R + 2 * MR * (kLdKeys + 8)) * 2 + (size_t)4 * MR * (kLdKeys + 4) * 4 + 3 * MR * 4;
}

bool latent_decode_serves(const TpxLatentAttn& a) {
  if (a.f32 || a.lat || a.S != 1 || a.R % 16 != 8 || a.krp % 16 || a.krp > 512 || a.R > 648 || a.past >= (1ll << 30)) return false;
  const int MR = a.heads <= 16 ? 16 : 32;
  const size_t smem = ld_smem_bytes(MR, (int)a.R);
  return smem <= 225 * 1024 && (size_t)MR * a.krp * 4 <= (size_t)kLdStages * kLdKeys * a.R * 2 && (((uintptr_t)a.qa | (uintptr_t)a.ol) & 15) == 0;
}

template <int MT, int CW, int KS>
static int latent_decode_launch(const TpxLatentAttn& a, cudaStream_t st) {
  const size_t smem = ld_smem_bytes(MT * 16, (int)a.R);
  static bool opted[16] = {};
  static int resident[9] = {};  // clusters of each size that fit the device at once (largest shared memory of this kernel)
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 16 || !opted[dev]) {
    TPX_CUDA_OK(cudaFuncSetAttribute(latent_decode_kernel<MT, CW, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  const int64_t groups = (a.heads + MT * 16 - 1) / (MT * 16), items = a.B * groups;
  // keys that may be in the window (planning only; the kernel reads the count itself)
  int64_t keys = a.npages * 32 < a.window ? a.npages * 32 : a.window;
  if (!a.dev_len && a.past + 1 < keys) keys = a.past + 1;
  const int64_t tiles = (keys + kLdKeys - 1) / kLdKeys;
  TPX_REQUIRE(a.npages < (1ll << 30), TPX_ERR_UNSUPPORTED, "latent decode: page table too long");
  cudaLaunchConfig_t cfg = {};
  cfg.blockDim = dim3(kLdThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = knobs().pdl;
  cfg.attrs = attr;
  int splits = tiles < 8 ? (int)tiles : 8;
  for (; splits > 1; splits--) {  // as many CTAs per sequence as run at once
    if (items * splits > sm_count()) continue;
    if (!resident[splits]) {
      cfg.gridDim = dim3((unsigned)splits, 1);
      cfg.numAttrs = 1;
      attr[0].val.clusterDim.x = (unsigned)splits;
      int n = 0;
      TPX_CUDA_OK(cudaOccupancyMaxActiveClusters(&n, latent_decode_kernel<MT, CW, KS>, &cfg));
      resident[splits] = n > 0 ? n : -1;
    }
    if (resident[splits] >= items) break;
  }
  if (splits < 1) splits = 1;
  attr[0].val.clusterDim.x = (unsigned)splits;
  cfg.gridDim = dim3((unsigned)(a.B * splits), (unsigned)groups);
  cfg.numAttrs = 2;
  count_launch();
  TPX_CUDA_OK(cudaLaunchKernelEx(&cfg, latent_decode_kernel<MT, CW, KS>, a, splits));
  return TPX_OK;
}

int latent_decode(const TpxLatentAttn& a, cudaStream_t st) {
  const bool one = a.heads <= 16;
  if (a.krp <= 128 && a.R <= 200) return one ? latent_decode_launch<1, 2, 3>(a, st) : latent_decode_launch<2, 2, 3>(a, st);
  if (a.krp <= 256 && a.R <= 328) return one ? latent_decode_launch<1, 4, 5>(a, st) : latent_decode_launch<2, 4, 5>(a, st);
  if (a.R <= 584) return one ? latent_decode_launch<1, 8, 9>(a, st) : latent_decode_launch<2, 8, 9>(a, st);
  return one ? latent_decode_launch<1, 8, 10>(a, st) : latent_decode_launch<2, 8, 10>(a, st);
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_latent_decode_status(void* stream, unsigned* status_host) {
  TPX_REQUIRE(status_host, TPX_ERR_ARG, "latent_decode_status: null pointer");
  static void* ptrs[64] = {};
  int dev = 0;
  TPX_CUDA_OK(cudaGetDevice(&dev));
  TPX_REQUIRE(dev >= 0 && dev < 64, TPX_ERR_UNSUPPORTED, "latent_decode_status: device index %d out of range", dev);
  if (!ptrs[dev]) TPX_CUDA_OK(cudaGetSymbolAddress(&ptrs[dev], g_latent_dec_err));
  TPX_CUDA_OK(cudaMemcpyAsync(status_host, ptrs[dev], 4, cudaMemcpyDeviceToHost, (cudaStream_t)stream));
  TPX_CUDA_OK(cudaMemsetAsync(ptrs[dev], 0, 4, (cudaStream_t)stream));
  TPX_CUDA_OK(cudaStreamSynchronize((cudaStream_t)stream));
  return TPX_OK;
}
