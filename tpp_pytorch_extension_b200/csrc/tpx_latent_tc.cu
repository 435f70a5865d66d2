// Prefill of latent attention on the 5th-generation tensor cores: keys and values of the call's tokens (and of the cached
// tokens still in the window) are expanded from the latents by one linear, then a flash-attention kernel with a sliding
// window, a value size of its own and the per-head output gate in its epilogue.
//
//   S = Q.K^T   A = 128 query tokens of one head, B = 128 keys; the contraction runs over 64-wide slabs: the plain part
//               (padded with zeros by the copies' bounds), then the rotated part, whose keys all heads share
//   T = P.V     A = P in tensor memory, B = 128 keys x vdim read MN-major
// The attention weights stay 32-bit in effect: P is written as two bf16 terms (hi + what hi leaves out) and both are
// multiplied with V. P takes the place of its scores in tensor memory (64 + 64 columns): the four warps that share a
// quarter's rows have all read their scores when they meet to exchange the row maxima.
//   warp 0   : TMA producer (Q once, then K and V tiles into two stages)
//   warp 1   : tensor memory, MMA issue: S of tile j+1 before P.V of tile j
//   warps 2-17: softmax and output, four warps per 32-row quarter (32 keys and vdim/4 output columns each)
#include "tpx_hybrid.cuh"
#include "tpx_tc_ptx.cuh"

namespace tpx {

static __device__ unsigned g_latent_tc_err;  // set when a bounded wait gave up; read and cleared by tpx_latent_tc_status

struct LatTcParams {
  const float* gate;  // [B*S][heads]
  const int* start;
  uint16_t* out;      // [B*S][ldo]
  long long ldo, past;
  int S, L, heads, dim, vdim, window;
  float scale;
};

// QS slabs of 64 for queries and keys (NS of them plain, the rest rotated), VS for values
template <int QS, int VS>
struct LtCfg {
  static constexpr int SLAB = 128 * 128;  // 128 rows x 64 bf16
  static constexpr int Q_BYTES = QS * SLAB, K_BYTES = QS * SLAB, V_BYTES = VS * SLAB, STAGE = K_BYTES + V_BYTES;
  static constexpr size_t SMEM = Q_BYTES + 2 * STAGE + 1024;
  static constexpr uint32_t COL_S = 0, COL_T = 256;
};

__device__ __forceinline__ void lt_tma_3d(uint32_t dst, const CUtensorMap* map, int c0, int c1, int c2, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(dst),
               "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void lt_mma_ss(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile("{ .reg .pred p; setp.ne.b32 p, %4, 0;\n  tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }" ::"r"(d), "l"(a), "l"(b),
               "r"(idesc), "r"(acc)
               : "memory");
}
__device__ __forceinline__ void lt_mma_ts(uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile("{ .reg .pred p; setp.ne.b32 p, %4, 0;\n  tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p; }" ::"r"(d), "r"(a), "l"(b),
               "r"(idesc), "r"(acc)
               : "memory");
}
__device__ __forceinline__ uint64_t lt_desc_mn(uint32_t saddr, uint32_t lbo) {  // as the values of tpx_attn_tc.cu
  return (uint64_t)((saddr & 0x3FFFFu) >> 4) | ((uint64_t)(lbo >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void lt_ld_x32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
        "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]),
        "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]),
        "=r"(r[31])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void lt_st_x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr), "r"(r[0]),
      "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]),
      "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ float lt_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t lt_pack(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

constexpr int kLtThreads = 64 + 512;

template <int QS, int VS>
__global__ void __launch_bounds__(kLtThreads, 1)
latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmR,
                      const __grid_constant__ CUtensorMap tmV, LatTcParams p, int NS) {
  using C = LtCfg<QS, VS>;
  extern __shared__ unsigned char lt_smem_raw[];
  __shared__ __align__(8) unsigned long long q_full, kv_full[2], kv_empty[2], s_full[2], p_full[2], o_full, o_free;
  __shared__ uint32_t tmem_holder;
  __shared__ float xmax[2][4][128];

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t smem_base = (tc_smem_u32(lt_smem_raw) + 1023u) & ~1023u;
  const uint32_t q_s = smem_base, kv_s = smem_base + C::Q_BYTES;
  const int head = blockIdx.x % p.heads, b = blockIdx.x / p.heads;
  const int chunk = (int)gridDim.y - 1 - (int)blockIdx.y;
  const int s0 = chunk * 128;

  if (threadIdx.x == 0) {
    tc_mbar_init(tc_smem_u32(&q_full), 1);
    for (int s = 0; s < 2; s++) {
      tc_mbar_init(tc_smem_u32(&kv_full[s]), 1);
      tc_mbar_init(tc_smem_u32(&kv_empty[s]), 1);
      tc_mbar_init(tc_smem_u32(&s_full[s]), 1);
      tc_mbar_init(tc_smem_u32(&p_full[s]), kLtThreads - 64);
    }
    tc_mbar_init(tc_smem_u32(&o_full), 1);
    tc_mbar_init(tc_smem_u32(&o_free), kLtThreads - 64);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tc_smem_u32(&tmem_holder)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_holder;
  pdl_trigger();
  pdl_wait();

  // key rows are indices into the buffer [L] of sequence b; query token s sits at row s + L - S
  const int back = p.L - p.S;
  const long long base = p.past - back;  // token index of row 0
  const int first = p.start ? max(0, (int)((long long)p.start[b] - base)) : 0;
  const int last_s = min(p.S, s0 + 128) - 1;
  const int kmin = max(first, s0 + back - p.window + 1);
  const int kmax = last_s + back + 1;
  const int j0 = max(kmin, 0) / 128;
  const int ntiles = kmax > kmin ? (kmax + 127) / 128 - j0 : 0;

  if (warp == 0) {
    if (lane == 0) {
      tc_mbar_expect_tx(tc_smem_u32(&q_full), C::Q_BYTES);
#pragma unroll
      for (int h = 0; h < QS; h++)
        lt_tma_3d(q_s + h * C::SLAB, &tmQ, h < NS ? h * 64 : p.dim + (h - NS) * 64, head, b * p.S + s0, tc_smem_u32(&q_full));
      for (int j = 0; j < ntiles; j++) {
        const int s = j & 1;
        if (j >= 2 && !tc_wait(tc_smem_u32(&kv_empty[s]), (uint32_t)(((j >> 1) - 1) & 1))) { atomicExch(&g_latent_tc_err, 2u); break; }
        const uint32_t st = kv_s + (uint32_t)s * C::STAGE;
        const uint32_t bar = tc_smem_u32(&kv_full[s]);
        const int row = b * p.L + (j0 + j) * 128;
        tc_mbar_expect_tx(bar, C::STAGE);
#pragma unroll
        for (int h = 0; h < QS; h++) {
          if (h < NS) lt_tma_3d(st + h * C::SLAB, &tmK, h * 64, head, row, bar);
          else tc_tma_2d(st + h * C::SLAB, &tmR, (h - NS) * 64, row, bar);
        }
#pragma unroll
        for (int h = 0; h < VS; h++) lt_tma_3d(st + C::K_BYTES + h * C::SLAB, &tmV, h * 64, head, row, bar);
      }
      // a call may end with no tile at all (padding only): the query copy must still have landed before the block exits
      if (!tc_wait(tc_smem_u32(&q_full), 0)) atomicExch(&g_latent_tc_err, 9u);
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 3) << 17) | ((128u >> 4) << 24);
      const uint32_t idesc_t = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(VS * 64 >> 3) << 17) | ((128u >> 4) << 24);
      bool ok = tc_wait(tc_smem_u32(&q_full), 0);
      if (!ok) atomicExch(&g_latent_tc_err, 3u);
      auto issue_s = [&](int j) -> bool {
        const int s = j & 1;
        if (!tc_wait(tc_smem_u32(&kv_full[s]), (uint32_t)((j >> 1) & 1))) { atomicExch(&g_latent_tc_err, 4u); return false; }
        tc_fence_after();
        const uint32_t ks = kv_s + (uint32_t)s * C::STAGE;
#pragma unroll
        for (int kk = 0; kk < QS * 4; kk++) {
          const uint32_t koff = (uint32_t)(kk >> 2) * C::SLAB + (uint32_t)(kk & 3) * 32;
          lt_mma_ss(tmem + C::COL_S + s * 128, tc_smem_desc(q_s + koff), tc_smem_desc(ks + koff), idesc_s, kk > 0 ? 1u : 0u);
        }
        tc_commit(tc_smem_u32(&s_full[s]));
        return true;
      };
      if (ok && ntiles > 0) ok = issue_s(0);
      for (int j = 0; ok && j < ntiles; j++) {
        const int s = j & 1;
        // the buffer of S_{j+1} held P_{j-1}: its P.V was issued before, and MMAs run in order
        if (j + 1 < ntiles && !issue_s(j + 1)) break;
        if (!tc_wait(tc_smem_u32(&p_full[s]), (uint32_t)((j >> 1) & 1))) { atomicExch(&g_latent_tc_err, 5u); break; }
        if (j > 0 && !tc_wait(tc_smem_u32(&o_free), (uint32_t)((j - 1) & 1))) { atomicExch(&g_latent_tc_err, 6u); break; }
        tc_fence_after();
        const uint32_t vs = kv_s + (uint32_t)s * C::STAGE + C::K_BYTES;
#pragma unroll
        for (int kk = 0; kk < 16; kk++)  // 8 steps of 16 keys with the leading terms of P, then 8 with what they left out
          lt_mma_ts(tmem + C::COL_T, tmem + C::COL_S + s * 128 + kk * 8, lt_desc_mn(vs + (kk & 7) * 2048, C::SLAB), idesc_t, kk > 0 ? 1u : 0u);
        tc_commit(tc_smem_u32(&o_full));
        tc_commit(tc_smem_u32(&kv_empty[s]));
      }
    }
    __syncwarp();
  } else {
    constexpr int HP = VS * 16;
    const int sub = warp & 3, part = (warp - 2) >> 2;
    const uint32_t lane_base = ((uint32_t)(sub * 32)) << 16;
    const int rl = sub * 32 + lane;
    const int s_tok = s0 + rl;
    const bool live = s_tok < p.S;
    const int khi = live ? s_tok + back + 1 : 0;                                  // keys [klo, khi) are visible
    const int klo = live ? max(first, s_tok + back - p.window + 1) : 0;
    const float sc2 = p.scale * 1.4426950408889634f;
    float o[HP];
#pragma unroll
    for (int i = 0; i < HP; i++) o[i] = 0.0f;
    float m_run = -INFINITY, l_run = 0.0f, alpha_prev = 1.0f;
    bool dead = false;
    auto accumulate = [&](int t, float alpha) {
      if (!tc_wait(tc_smem_u32(&o_full), (uint32_t)(t & 1))) { atomicExch(&g_latent_tc_err, 7u); dead = true; return; }
      tc_fence_after();
      uint32_t v[HP];
      if (HP == 32) lt_ld_x32(tmem + lane_base + C::COL_T + part * HP, reinterpret_cast<uint32_t(&)[32]>(v));
      else tc_ld_x16(tmem + lane_base + C::COL_T + part * HP, reinterpret_cast<uint32_t(&)[16]>(v));
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int i = 0; i < HP; i++) o[i] = fmaf(o[i], alpha, __uint_as_float(v[i]));
      tc_fence_before();
      tc_mbar_arrive(tc_smem_u32(&o_free));
    };
    for (int j = 0; j < ntiles && !dead; j++) {
      const int s = j & 1;
      if (!tc_wait(tc_smem_u32(&s_full[s]), (uint32_t)((j >> 1) & 1))) { atomicExch(&g_latent_tc_err, 8u); dead = true; break; }
      tc_fence_after();
      const int k0 = (j0 + j) * 128 + part * 32;
      uint32_t v[32];
      lt_ld_x32(tmem + lane_base + C::COL_S + s * 128 + part * 32, v);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      float x[32];
      if (k0 >= klo && k0 + 32 <= khi) {
#pragma unroll
        for (int i = 0; i < 32; i++) x[i] = __uint_as_float(v[i]) * sc2;
      } else {
#pragma unroll
        for (int i = 0; i < 32; i++) x[i] = (k0 + i >= klo && k0 + i < khi) ? __uint_as_float(v[i]) * sc2 : -INFINITY;
      }
      float t4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < 32; i++) t4[i & 3] = fmaxf(t4[i & 3], x[i]);
      xmax[s][part][rl] = fmaxf(fmaxf(t4[0], t4[1]), fmaxf(t4[2], t4[3]));
      tc_fence_before();
      asm volatile("bar.sync %0, 128;" ::"r"(1 + sub) : "memory");  // the four warps of this quarter: their scores are in registers
      tc_fence_after();
      const float tmax = fmaxf(fmaxf(xmax[s][0][rl], xmax[s][1][rl]), fmaxf(xmax[s][2][rl], xmax[s][3][rl]));
      const float m_new = fmaxf(m_run, tmax);
      const float alpha = (m_new == -INFINITY) ? 1.0f : lt_ex2(m_run - m_new);
      const float mref = (m_new == -INFINITY) ? 0.0f : m_new;
      float l4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      uint32_t hi[16], lo[16];
#pragma unroll
      for (int i = 0; i < 32; i += 2) {
        const float e0 = lt_ex2(x[i] - mref), e1 = lt_ex2(x[i + 1] - mref);
        l4[(i >> 1) & 3] += e0 + e1;
        const uint32_t h = lt_pack(e0, e1);
        hi[i >> 1] = h;
        lo[i >> 1] = lt_pack(e0 - __uint_as_float(h << 16), e1 - __uint_as_float(h & 0xffff0000u));
      }
      lt_st_x16(tmem + lane_base + C::COL_S + s * 128 + part * 16, hi);
      lt_st_x16(tmem + lane_base + C::COL_S + s * 128 + 64 + part * 16, lo);
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      tc_fence_before();
      tc_mbar_arrive(tc_smem_u32(&p_full[s]));
      l_run = l_run * alpha + ((l4[0] + l4[1]) + (l4[2] + l4[3]));
      m_run = m_new;
      if (j > 0) accumulate(j - 1, alpha_prev);
      alpha_prev = alpha;
    }
    if (!dead && ntiles > 0) accumulate(ntiles - 1, alpha_prev);
    xmax[0][part][rl] = l_run;
    asm volatile("bar.sync %0, 128;" ::"r"(1 + sub) : "memory");
    const float l_tot = (xmax[0][0][rl] + xmax[0][1][rl]) + (xmax[0][2][rl] + xmax[0][3][rl]);
    if (live && !dead) {
      const long long row = (long long)b * p.S + s_tok;
      const float inv = l_tot > 0.0f ? p.gate[row * p.heads + head] / l_tot : 0.0f;
      uint16_t* dst = p.out + row * p.ldo + (long long)head * p.vdim + part * HP;
#pragma unroll
      for (int i = 0; i < HP; i += 8) {
        if (part * HP + i < p.vdim) {
          uint32_t w[4];
#pragma unroll
          for (int u = 0; u < 4; u++) w[u] = lt_pack(o[i + 2 * u] * inv, o[i + 2 * u + 1] * inv);
          *reinterpret_cast<uint4*>(dst + i) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
  }
}

// rotation of the last rot_dim values of every head of q, in place: a warp per (token, head)
__global__ void __launch_bounds__(256) latent_rotate_kernel(__nv_bfloat16* __restrict__ q, const float2* __restrict__ cs, int64_t items, int heads,
                                                            int dim, int rot, int64_t ldq) {
  pdl_trigger();
  pdl_wait();
  const int64_t item = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= items) return;
  const int64_t row = item / heads;
  const int head = (int)(item % heads);
  __nv_bfloat162* x = reinterpret_cast<__nv_bfloat162*>(q + row * ldq + (int64_t)head * (dim + rot) + dim);
  for (int i = threadIdx.x & 31; i < rot / 2; i += 32) {
    const float2 r = cs[row * (rot / 2) + i], v = __bfloat1622float2(x[i]);
    x[i] = __floats2bfloat162_rn(v.x * r.x - v.y * r.y, v.y * r.x + v.x * r.y);
  }
}

typedef CUresult (*LtEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                               const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static int lt_map(CUtensorMap* m, const void* base, int rank, const uint64_t* dims, const uint64_t* strides_bytes) {
  static LtEncodeFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &ptr, 12000, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<LtEncodeFn>(ptr);
  }
  TPX_REQUIRE(fn, TPX_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
  cuuint64_t g[3], st[2];
  cuuint32_t box[3] = {64, 1, 128}, es[3] = {1, 1, 1};
  for (int i = 0; i < rank; i++) g[i] = dims[i];
  for (int i = 0; i + 1 < rank; i++) st[i] = strides_bytes[i];
  if (rank == 2) box[1] = 128;
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(base), g, st, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  TPX_REQUIRE(r == CUDA_SUCCESS, TPX_ERR_CUDA, "latent prefill: cuTensorMapEncodeTiled failed with %d", (int)r);
  return TPX_OK;
}

template <int QS, int VS>
static int lt_launch(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& r, const CUtensorMap& v, const LatTcParams& p, int NS, int64_t B,
                     cudaStream_t st) {
  using C = LtCfg<QS, VS>;
  static bool opted[16] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 16 || !opted[dev]) {
    TPX_CUDA_OK(cudaFuncSetAttribute(latent_attn_tc_kernel<QS, VS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  TPX_CUDA_OK(launch_pdl(latent_attn_tc_kernel<QS, VS>, dim3((unsigned)(B * p.heads), (unsigned)((p.S + 127) / 128)), dim3(kLtThreads), C::SMEM, st, q, k,
                         r, v, p, NS));
  return TPX_OK;
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_latent_prefill_serves(int64_t dim, int64_t rot_dim, int64_t vdim) {
  if (dim <= 0 || rot_dim < 0 || vdim <= 0 || dim % 8 || rot_dim % 8 || vdim % 8 || vdim > 128) return 0;
  const int64_t slabs = (dim + 63) / 64 + (rot_dim + 63) / 64;
  return slabs <= 3;
}

extern "C" int tpx_latent_prefill(const TpxLatentPrefill* a, void* stream) {
  TPX_REQUIRE(a, TPX_ERR_ARG, "latent_prefill: null argument block");
  TPX_REQUIRE(tpx_latent_prefill_serves(a->dim, a->rot_dim, a->vdim), TPX_ERR_UNSUPPORTED, "latent_prefill: head sizes %ld + %ld, %ld are not served",
              (long)a->dim, (long)a->rot_dim, (long)a->vdim);
  TPX_REQUIRE(a->B >= 0 && a->S >= 0 && a->L >= a->S && a->heads > 0 && a->window > 0 && a->past >= a->L - a->S, TPX_ERR_ARG, "latent_prefill: bad shape");
  TPX_REQUIRE(a->L - a->S >= (a->window - 1 < a->past ? a->window - 1 : a->past), TPX_ERR_ARG, "latent_prefill: the keys of the window are not there");
  if (a->B == 0 || a->S == 0) return TPX_OK;
  TPX_REQUIRE(a->q && a->kv && a->lat && a->gate && a->out && (a->rot_dim == 0 || a->cos_sin), TPX_ERR_ARG, "latent_prefill: null pointer");
  TPX_REQUIRE(a->ldq % 8 == 0 && a->ldkv % 8 == 0 && a->ldo % 8 == 0 && a->R % 8 == 0 && a->krp % 8 == 0 && a->ldq >= a->heads * (a->dim + a->rot_dim) &&
                  a->ldkv >= a->heads * (a->dim + a->vdim) && a->ldo >= a->heads * a->vdim, TPX_ERR_ARG, "latent_prefill: bad leading dimension");
  TPX_REQUIRE((((uintptr_t)a->q | (uintptr_t)a->kv | (uintptr_t)a->lat | (uintptr_t)a->out) & 15) == 0, TPX_ERR_ARG, "latent_prefill: misaligned pointer");
  TPX_REQUIRE(a->B * a->heads < (1ll << 31) && a->B * a->L < (1ll << 31) && a->S <= 65535ll * 128 && a->window < (1ll << 30), TPX_ERR_UNSUPPORTED,
              "latent_prefill: shape too large");
  cudaStream_t st = (cudaStream_t)stream;
  const int64_t items = a->B * a->S * a->heads;
  if (a->rot_dim)
    TPX_CUDA_OK(launch_pdl(latent_rotate_kernel, dim3((unsigned)((items + 7) / 8)), dim3(256), 0, st, (__nv_bfloat16*)a->q,
                           (const float2*)a->cos_sin, items, (int)a->heads, (int)a->dim, (int)a->rot_dim, a->ldq));
  CUtensorMap mq, mk, mr, mv;
  const uint64_t H = (uint64_t)a->heads, hd = (uint64_t)(a->dim + a->rot_dim);
  const uint64_t qd[3] = {hd, H, (uint64_t)(a->B * a->S)}, qs[2] = {hd * 2, (uint64_t)a->ldq * 2};
  const uint64_t kd[3] = {(uint64_t)a->dim, H, (uint64_t)(a->B * a->L)}, ks[2] = {(uint64_t)a->dim * 2, (uint64_t)a->ldkv * 2};
  const uint64_t vd[3] = {(uint64_t)a->vdim, H, (uint64_t)(a->B * a->L)}, vs[2] = {(uint64_t)a->vdim * 2, (uint64_t)a->ldkv * 2};
  const uint64_t rd[2] = {(uint64_t)(a->rot_dim ? a->rot_dim : 8), (uint64_t)(a->B * a->L)}, rs[1] = {(uint64_t)a->R * 2};
  int rc = lt_map(&mq, a->q, 3, qd, qs);
  if (!rc) rc = lt_map(&mk, a->kv, 3, kd, ks);
  if (!rc) rc = lt_map(&mv, (const uint16_t*)a->kv + H * a->dim, 3, vd, vs);
  if (!rc) rc = lt_map(&mr, a->rot_dim ? (const uint16_t*)a->lat + a->krp : (const uint16_t*)a->lat, 2, rd, rs);
  if (rc) return rc;
  LatTcParams p = {a->gate, a->start, (uint16_t*)a->out, (long long)a->ldo, (long long)a->past, (int)a->S, (int)a->L, (int)a->heads, (int)a->dim,
                   (int)a->vdim, (int)a->window, a->scale};
  const int NS = (int)((a->dim + 63) / 64), QS = NS + (int)((a->rot_dim + 63) / 64), VS = (int)((a->vdim + 63) / 64);
  switch (QS * 10 + VS) {
    case 11: return lt_launch<1, 1>(mq, mk, mr, mv, p, NS, a->B, st);
    case 12: return lt_launch<1, 2>(mq, mk, mr, mv, p, NS, a->B, st);
    case 21: return lt_launch<2, 1>(mq, mk, mr, mv, p, NS, a->B, st);
    case 22: return lt_launch<2, 2>(mq, mk, mr, mv, p, NS, a->B, st);
    case 31: return lt_launch<3, 1>(mq, mk, mr, mv, p, NS, a->B, st);
    default: return lt_launch<3, 2>(mq, mk, mr, mv, p, NS, a->B, st);
  }
}

extern "C" int tpx_latent_tc_status(void* stream, unsigned* status_host) {
  TPX_REQUIRE(status_host, TPX_ERR_ARG, "latent_tc_status: null pointer");
  static void* ptrs[64] = {};
  int dev = 0;
  TPX_CUDA_OK(cudaGetDevice(&dev));
  TPX_REQUIRE(dev >= 0 && dev < 64, TPX_ERR_UNSUPPORTED, "latent_tc_status: device index %d out of range", dev);
  if (!ptrs[dev]) TPX_CUDA_OK(cudaGetSymbolAddress(&ptrs[dev], g_latent_tc_err));
  TPX_CUDA_OK(cudaMemcpyAsync(status_host, ptrs[dev], 4, cudaMemcpyDeviceToHost, (cudaStream_t)stream));
  TPX_CUDA_OK(cudaMemsetAsync(ptrs[dev], 0, 4, (cudaStream_t)stream));
  TPX_CUDA_OK(cudaStreamSynchronize((cudaStream_t)stream));
  return TPX_OK;
}
