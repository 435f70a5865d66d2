// Decoding with chunked differential attention in bf16: one token per sequence against the pages of its chunk.
//
// A thread-block cluster per (sequence, key / value head, group of 8 query heads); its CTAs share the chunk's pages, and a CTA's
// warps take them in turn, each with two stages of its own filled by one bulk copy per page (32 rows of both keys and the value,
// contiguous; rows carry 8 elements of padding and lie in different banks). The 16 rows of an MMA are map 1 of the 8 heads,
// then map 2: the products with map 1's keys have zeros in the lower rows, those with map 2's in the upper, so one accumulator
// holds both maps and a thread the two maps of one head. The cap bounds the scores, so exp takes no maximum off and everything
// that warps and CTAs hold is put together by adding. Weights are multiplied as two bf16 terms. The call's own token is not
// read from the cache: the warp with the last page puts it into its copy, and into the page.
#include "tpx_hybrid.cuh"
#include "tpx_tc_ptx.cuh"

namespace tpx {

static __device__ unsigned g_diff_dec_err;  // set when a bounded wait gave up; read and cleared by tpx_diff_status
constexpr int kDdMaxWarps = 6, kDdStages = 2, kDdHeads = 8;

__device__ __forceinline__ void dd_ldm_x4(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void dd_ldm_x4t(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void dd_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t dd_pack(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float dd_ld_cluster(uint32_t saddr, uint32_t rank) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(tc_mapa(saddr, rank)) : "memory");
  return v;
}

// KS: 16-wide steps of one map's key, at most; NT: 8-wide value tiles, at most
template <int KS, int NT>
__global__ void __launch_bounds__(kDdMaxWarps * 32, 1) diff_decode_kernel(TpxDiffAttn p, int splits, int groups) {
  constexpr int VC = NT * 8;
  extern __shared__ __align__(16) unsigned char dd_smem[];
  __shared__ __align__(8) unsigned long long full[kDdMaxWarps][kDdStages];
  __shared__ float sl[kDdMaxWarps][16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int R = (int)p.R, dim = (int)p.dim, vdim = (int)p.vdim, dp = (dim + 15) / 16 * 16, ks = dp / 16;
  const int rank = blockIdx.x % splits, b = blockIdx.x / splits;
  const int g = blockIdx.y / groups, grp = blockIdx.y % groups, rq = (int)(p.heads / p.kv_heads);
  const int nh = min(kDdHeads, rq - grp * kDdHeads), h0 = g * rq + grp * kDdHeads;
  uint16_t* mine = reinterpret_cast<uint16_t*>(dd_smem) + (size_t)warp * kDdStages * 32 * R;
  pdl_trigger();
  if (lane == 0) {
    for (int i = 0; i < kDdStages; i++) tc_mbar_init(tc_smem_u32(&full[warp][i]), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  __syncwarp();
  pdl_wait();
  const int64_t t = p.dev_len ? *p.dev_len : p.past, start = p.start ? p.start[b] : 0;
  const int64_t lo = t < start ? t : start + (t - start) / p.chunk * p.chunk;
  const int blk0 = (int)(lo / 32), tiles = (int)(t / 32) - blk0 + 1;  // tile i: page blk0 + i
  const int i0 = (int)((long long)tiles * rank / splits), i1 = (int)((long long)tiles * (rank + 1) / splits);
  const int np = (int)p.npages;
  auto page = [&](int i) { return reinterpret_cast<uint16_t*>(__ldg(p.pages + (blk0 + i) % np)) + ((int64_t)b * p.kv_heads + g) * 32 * R; };
  auto fetch = [&](int i, int st) {  // one lane
    const uint32_t bar = tc_smem_u32(&full[warp][st]);
    tc_mbar_expect_tx(bar, (uint32_t)(32 * R * 2));
    tc_bulk_g2s(tc_smem_u32(mine + (size_t)st * 32 * R), page(i), (uint32_t)(32 * R * 2), bar);
  };
  if (lane == 0)
    for (int s = 0; s < kDdStages; s++)
      if (i0 + warp + s * warps < i1) fetch(i0 + warp + s * warps, s);
  const uint16_t* pr = reinterpret_cast<const uint16_t*>(p.proj) + (int64_t)b * p.ldp;
  // queries as MMA operands: row lane / 4 is head h0 + lane / 4
  uint32_t qf[2][KS][2];
  const int hl = lane >> 2;
#pragma unroll
  for (int m = 0; m < 2; m++)
#pragma unroll
    for (int k = 0; k < KS; k++)
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int c = k * 16 + e * 8 + (lane & 3) * 2;  // dim is even
        qf[m][k][e] = hl < nh && c < dim ? *reinterpret_cast<const uint32_t*>(pr + p.q_col + ((int64_t)(h0 + hl) * 2 + m) * dim + c) : 0u;
      }
  float o[NT][4], l[2] = {0.0f, 0.0f};
#pragma unroll
  for (int i = 0; i < NT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
  const float zc = p.scale / p.softcap * 2.8853900817779268f, tc = p.softcap * 1.4426950408889634f;
  bool dead = false;
  int it = 0;
  for (int i = i0 + warp; i < i1; i += warps, it++) {
    const int st = it % kDdStages;
    uint16_t* kt = mine + (size_t)st * 32 * R;
    if (!dead && !tc_wait(tc_smem_u32(&full[warp][st]), (uint32_t)((it / kDdStages) & 1))) {
      dead = true;
      if (lane == 0) atomicExch(&g_diff_dec_err, 1u);
    }
    const int64_t k0 = (int64_t)(blk0 + i) * 32;
    const int from = (int)max((int64_t)0, lo - k0), to = (int)min((int64_t)31, t - k0);  // keys from .. to count
    if (from > 0 || to < 31 || i == tiles - 1) {  // what lies outside may be anything; the last key is the call's own
      for (int q = lane; q < 32 * (R / 8); q += 32) {
        const int key = q / (R / 8);
        if (key < from || key > to) *reinterpret_cast<uint4*>(kt + q * 8) = make_uint4(0, 0, 0, 0);
      }
      __syncwarp();
      if (i == tiles - 1) {
        uint16_t* dst = kt + to * R;
        uint16_t* keep = page(i) + to * R;
        for (int c = lane; c < R; c += 32) {
          const int m = c / dp, cc = c % dp;
          uint16_t v = 0;
          if (m < 2) {
            if (cc < dim) v = pr[p.k_col + ((int64_t)g * 2 + m) * dim + cc];
          } else if (c - 2 * dp < vdim) {
            v = pr[p.v_col + (int64_t)g * vdim + c - 2 * dp];
          }
          dst[c] = v;
          if (grp == 0) keep[c] = v;
        }
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // a later copy into this stage comes after these writes
      __syncwarp();
    }
    float sc[4][4];
#pragma unroll
    for (int n = 0; n < 4; n++) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.0f;
    const uint32_t kb = tc_smem_u32(kt + ((lane & 7) + ((lane >> 4) & 1) * 8) * R + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int m = 0; m < 2; m++)
#pragma unroll
      for (int k = 0; k < KS; k++) {
        const uint32_t at = kb + (uint32_t)(m * ks + min(k, ks - 1)) * 32;  // steps the key does not have meet zero queries
#pragma unroll
        for (int n = 0; n < 4; n += 2) {
          uint32_t kf[4];
          dd_ldm_x4(at + n * 8 * R * 2, kf);
          const uint32_t q0 = qf[m][k][0], q1 = qf[m][k][1];
          dd_mma(sc[n], m ? 0u : q0, m ? q0 : 0u, m ? 0u : q1, m ? q1 : 0u, kf[0], kf[1]);
          dd_mma(sc[n + 1], m ? 0u : q0, m ? q0 : 0u, m ? 0u : q1, m ? q1 : 0u, kf[2], kf[3]);
        }
      }
#pragma unroll
    for (int n = 0; n < 4; n++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int key = n * 8 + (lane & 3) * 2 + (e & 1);
        const float x = exp2f(fmaf(-2.0f * tc, __fdividef(1.0f, exp2f(sc[n][e] * zc) + 1.0f), tc));  // exp(softcap tanh(.))
        sc[n][e] = key >= from && key <= to ? x : 0.0f;
        l[e >> 1] += sc[n][e];
      }
    const uint32_t vb = tc_smem_u32(kt + (((lane >> 3) & 1) * 8 + (lane & 7)) * R + 2 * dp + (lane >> 4) * 8);
#pragma unroll
    for (int j = 0; j < 2; j++) {
      uint32_t hi[4], lw[4];
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const float x = sc[2 * j + (e >> 1)][(e & 1) * 2], y = sc[2 * j + (e >> 1)][(e & 1) * 2 + 1];
        hi[e] = dd_pack(x, y);
        lw[e] = dd_pack(x - __uint_as_float(hi[e] << 16), y - __uint_as_float(hi[e] & 0xffff0000u));
      }
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        uint32_t vf[4];
        dd_ldm_x4t(vb + (uint32_t)(j * 16 * R + min(n * 8, (vdim + 15) / 16 * 16 - 16)) * 2, vf);  // tiles beyond: dropped
        dd_mma(o[n], hi[0], hi[1], hi[2], hi[3], vf[0], vf[1]);
        dd_mma(o[n + 1], hi[0], hi[1], hi[2], hi[3], vf[2], vf[3]);
        dd_mma(o[n], lw[0], lw[1], lw[2], lw[3], vf[0], vf[1]);
        dd_mma(o[n + 1], lw[0], lw[1], lw[2], lw[3], vf[2], vf[3]);
      }
    }
    __syncwarp();
    if (lane == 0 && i + kDdStages * warps < i1) fetch(i + kDdStages * warps, st);
  }
  // sums over the warps, then over the cluster
#pragma unroll
  for (int h = 0; h < 2; h++) {
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
  }
  __syncthreads();  // the stages are free
  float* so = reinterpret_cast<float*>(dd_smem);  // [warps][16][VC]
  if ((lane & 3) == 0) { sl[warp][hl] = l[0]; sl[warp][hl + 8] = l[1]; }
#pragma unroll
  for (int i = 0; i < NT; i++) {
    *reinterpret_cast<float2*>(so + (size_t)(warp * 16 + hl) * VC + i * 8 + (lane & 3) * 2) = make_float2(o[i][0], o[i][1]);
    *reinterpret_cast<float2*>(so + (size_t)(warp * 16 + hl + 8) * VC + i * 8 + (lane & 3) * 2) = make_float2(o[i][2], o[i][3]);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < 16 * VC; i += blockDim.x) {
    float x = so[i];
    for (int w = 1; w < warps; w++) x += so[w * 16 * VC + i];
    so[i] = x;
  }
  if (threadIdx.x < 16) {
    float x = sl[0][threadIdx.x];
    for (int w = 1; w < warps; w++) x += sl[w][threadIdx.x];
    sl[0][threadIdx.x] = x;
  }
  __syncthreads();
  tc_cluster_sync();
  constexpr int CL = (VC + 31) / 32;
  for (int h = rank * warps + warp; h < nh; h += splits * warps) {
    float l1 = 0.0f, l2 = 0.0f, a1[CL] = {}, a2[CL] = {};
    for (int c = 0; c < splits; c++) {
      l1 += dd_ld_cluster(tc_smem_u32(&sl[0][h]), c);
      l2 += dd_ld_cluster(tc_smem_u32(&sl[0][h + 8]), c);
#pragma unroll
      for (int i = 0; i < CL; i++)
        if (lane + 32 * i < vdim) {
          a1[i] += dd_ld_cluster(tc_smem_u32(so + h * VC + lane + 32 * i), c);
          a2[i] += dd_ld_cluster(tc_smem_u32(so + (h + 8) * VC + lane + 32 * i), c);
        }
    }
    const float i1 = 1.0f / l1, i2 = p.lambda / l2;
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < CL; i++) {
      a1[i] = lane + 32 * i < vdim ? a1[i] * i1 - a2[i] * i2 : 0.0f;
      ss = fmaf(a1[i], a1[i], ss);
    }
    const float inv = p.mult / sqrtf(hy_warp_sum(ss) / (float)vdim + p.eps);
    uint16_t* out = reinterpret_cast<uint16_t*>(p.out) + (int64_t)b * p.ldo + (int64_t)(h0 + h) * vdim;
#pragma unroll
    for (int i = 0; i < CL; i++)
      if (lane + 32 * i < vdim) out[lane + 32 * i] = f32_to_bf16_bits(a1[i] * inv);
  }
  tc_cluster_sync();  // nobody leaves while its shared memory is being read
}

static int dd_warps(int64_t R) {
  const int64_t fit = (220 * 1024) / (kDdStages * 32 * R * 2);
  return fit > kDdMaxWarps ? kDdMaxWarps : (int)fit;
}

bool diff_decode_serves(const TpxDiffAttn& a) {
  return !a.f32 && a.S == 1 && diff_prefill_serves(a.dim, a.vdim, a.softcap) && a.ldp % 2 == 0 && a.q_col % 2 == 0 && a.npages < (1ll << 30) &&
         ((uintptr_t)a.proj & 3) == 0 && dd_warps(a.R) >= 1;
}

template <int KS, int NT>
static int dd_launch(const TpxDiffAttn& a, cudaStream_t st) {
  int warps = dd_warps(a.R);
  size_t smem = (size_t)warps * kDdStages * 32 * a.R * 2;
  static_assert(kDdStages * 32 * 2 >= 16 * 4, "the sums fit the stages");
  static bool opted[16] = {};
  static int resident[9] = {};  // clusters of each size that fit the device at once (largest shared memory of this kernel)
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 16 || !opted[dev]) {
    TPX_CUDA_OK(cudaFuncSetAttribute(diff_decode_kernel<KS, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  const int64_t rq = a.heads / a.kv_heads, groups = (rq + kDdHeads - 1) / kDdHeads, items = a.B * a.kv_heads * groups;
  // keys that the token may see (planning only; the kernel reads the count itself)
  int64_t keys = a.npages * 32 < a.chunk ? a.npages * 32 : a.chunk;
  if (!a.dev_len && a.past + 1 < keys) keys = a.past + 1;
  const int64_t tiles = (keys + 31) / 32;
  cudaLaunchConfig_t cfg = {};
  cfg.blockDim = dim3((unsigned)warps * 32);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = knobs().pdl;
  cfg.attrs = attr;
  int splits = tiles < 8 ? (int)tiles : 8;
  for (; splits > 1; splits--) {  // as many CTAs per item as run at once
    if (items * splits > sm_count()) continue;
    if (!resident[splits]) {
      cfg.gridDim = dim3((unsigned)splits, 1);
      cfg.numAttrs = 1;
      attr[0].val.clusterDim.x = (unsigned)splits;
      int n = 0;
      TPX_CUDA_OK(cudaOccupancyMaxActiveClusters(&n, diff_decode_kernel<KS, NT>, &cfg));
      resident[splits] = n > 0 ? n : -1;
    }
    if (resident[splits] >= items) break;
  }
  if (splits < 1) splits = 1;
  attr[0].val.clusterDim.x = (unsigned)splits;
  cfg.gridDim = dim3((unsigned)(a.B * splits), (unsigned)(a.kv_heads * groups));
  TPX_REQUIRE(a.kv_heads * groups <= 65535, TPX_ERR_UNSUPPORTED, "diff decode: too many heads");
  cfg.numAttrs = 2;
  count_launch();
  TPX_CUDA_OK(cudaLaunchKernelEx(&cfg, diff_decode_kernel<KS, NT>, a, splits, (int)groups));
  return TPX_OK;
}

template <int KS>
static int dd_values(const TpxDiffAttn& a, cudaStream_t st) {
  return a.vdim <= 32 ? dd_launch<KS, 4>(a, st) : a.vdim <= 64 ? dd_launch<KS, 8>(a, st) : dd_launch<KS, 16>(a, st);
}

int diff_decode(const TpxDiffAttn& a, cudaStream_t st) { return a.dim <= 32 ? dd_values<2>(a, st) : a.dim <= 64 ? dd_values<4>(a, st) : dd_values<8>(a, st); }

int diff_tc_status(cudaStream_t st, unsigned* host);

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_diff_status(void* stream, unsigned* status_host) {
  TPX_REQUIRE(status_host, TPX_ERR_ARG, "diff_status: null pointer");
  cudaStream_t st = (cudaStream_t)stream;
  static void* ptrs[64] = {};
  int dev = 0;
  TPX_CUDA_OK(cudaGetDevice(&dev));
  TPX_REQUIRE(dev >= 0 && dev < 64, TPX_ERR_UNSUPPORTED, "diff_status: device index %d out of range", dev);
  if (!ptrs[dev]) TPX_CUDA_OK(cudaGetSymbolAddress(&ptrs[dev], g_diff_dec_err));
  unsigned tc = 0;
  const int rc = diff_tc_status(st, &tc);
  if (rc) return rc;
  TPX_CUDA_OK(cudaMemcpyAsync(status_host, ptrs[dev], 4, cudaMemcpyDeviceToHost, st));
  TPX_CUDA_OK(cudaMemsetAsync(ptrs[dev], 0, 4, st));
  TPX_CUDA_OK(cudaStreamSynchronize(st));
  if (tc) *status_host = 16 + tc;
  return TPX_OK;
}
