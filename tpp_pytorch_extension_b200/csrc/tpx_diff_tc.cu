// Prefill of chunked differential attention on the 5th-generation tensor cores. A CTA owns 128 query tokens of one head and both
// of its maps; a map's scores come from keys of its own, the values are shared:
//   S_m = Q_m.K_m^T   A = 128 queries, B = 128 keys of map m, 64-wide slabs of the contraction (padded with zeros by the copies' bounds)
//   O_m += P_m.V      A = P_m in tensor memory, B = 128 keys x vdim read MN-major, accumulated in tensor memory over all tiles
// The cap bounds every score, |softcap tanh(..)| <= softcap, so exp needs no maximum taken off: nothing is rescaled, no row
// statistics are exchanged between tiles, and the outputs stay in tensor memory until the end. P is written as two bf16 terms (value
// and what rounding left out), both multiplied with V, so that the weights stay 32-bit in effect.
//   warp 0    : TMA producer, a ring of tiles in the order K_1, K_2, V
//   warp 1    : tensor memory, MMA issue: while the softmax warps of one map work, the other map's products run
//   warps 2-9 : map 1, warps 10-17: map 2; two warps per 32-row quarter, 64 keys of the tile each. A warp's scores and the P it
//               makes of them share the same columns, so that the warps of a map need not meet
// tanh is a polynomial where a warp's scores stay below the cap (|s| <= softcap), else by its exponential. At the end the sixteen
// warps put the two outputs together, norm the heads and store bf16.
#include "tpx_hybrid.cuh"
#include "tpx_tc_ptx.cuh"

namespace tpx {

static __device__ unsigned g_diff_tc_err;  // set when a bounded wait gave up; read and cleared by tpx_diff_status

constexpr float kDiffMaxCap = 64.0f;  // exp(+-64), summed over any number of keys, is far from the ends of fp32 and bf16

struct DiffTcParams {
  const int* start;
  uint16_t* out;
  long long ldo, past;
  int S, L, heads, group, vdim, chunk;  // group: query heads per key / value head
  float scale, softcap, lambda, mult, eps;
};

// DS slabs of 64 for one map's queries and keys, VS for values
template <int DS, int VS>
struct DtCfg {
  static constexpr int SLAB = 128 * 128;  // 128 rows x 64 bf16
  static constexpr int Q_BYTES = 2 * DS * SLAB, SLOT = (DS > VS ? DS : VS) * SLAB;
  static constexpr int FIT = (221 * 1024 - Q_BYTES) / SLOT, SLOTS = FIT > 6 ? 6 : FIT;
  static constexpr size_t SMEM = Q_BYTES + (size_t)SLOTS * SLOT + 1024;
  static constexpr uint32_t COL_S = 0, COL_O = 256;
  static_assert(SLOTS >= 4, "tiles in flight");
};

constexpr int kDtThreads = 64 + 512;

__device__ __forceinline__ void dt_tma_3d(uint32_t dst, const CUtensorMap* map, int c0, int c1, int c2, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(dst),
               "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void dt_tma_4d(uint32_t dst, const CUtensorMap* map, int c0, int c1, int c2, int c3, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5}], [%6];" ::"r"(dst),
               "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void dt_mma_ss(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile("{ .reg .pred p; setp.ne.b32 p, %4, 0;\n  tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }" ::"r"(d), "l"(a), "l"(b),
               "r"(idesc), "r"(acc)
               : "memory");
}
__device__ __forceinline__ void dt_mma_ts(uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile("{ .reg .pred p; setp.ne.b32 p, %4, 0;\n  tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p; }" ::"r"(d), "r"(a), "l"(b),
               "r"(idesc), "r"(acc)
               : "memory");
}
// values [key][vdim] as an MN-major operand: 128-byte rows of 64 values, 8-key groups 1024 bytes apart, the next 64 values lbo further
__device__ __forceinline__ uint64_t dt_desc_mn(uint32_t saddr, uint32_t lbo) {
  return (uint64_t)((saddr & 0x3FFFFu) >> 4) | ((uint64_t)(lbo >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void dt_ld_x32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
        "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]),
        "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]),
        "=r"(r[31])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void dt_st_x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr), "r"(r[0]),
      "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]),
      "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ float dt_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t dt_pack(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float2 dt_fma2(float2 a, float2 b, float2 c) {
  unsigned long long r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(r)
      : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)), "l"(*reinterpret_cast<unsigned long long*>(&c)));
  return *reinterpret_cast<float2*>(&r);
}
__device__ __forceinline__ float2 dt_mul2(float2 a, float2 b) {
  unsigned long long r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)));
  return *reinterpret_cast<float2*>(&r);
}
__device__ __forceinline__ float2 dt_two(float a) { return make_float2(a, a); }

// log2 of exp(softcap tanh(s / softcap)) for 32 raw scores; zc: score to s / softcap, uc: score to s log2(e), tc: softcap log2(e).
// tanh(z) / z on |z| <= 1 is a polynomial in z^2: the interpolant at the Chebyshev nodes of [0, 1], relative error below 1.3e-7.
__device__ __forceinline__ void dt_capped(uint32_t (&v)[32], float zc, float uc, float tc) {
  float b4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (int i = 0; i < 32; i += 2) b4[(i >> 1) & 3] = fmaxf(fmaxf(b4[(i >> 1) & 3], fabsf(__uint_as_float(v[i]))), fabsf(__uint_as_float(v[i + 1])));
  const float big = fmaxf(fmaxf(b4[0], b4[1]), fmaxf(b4[2], b4[3]));
  if (__any_sync(0xffffffffu, big * zc > 1.0f)) {
#pragma unroll
    for (int i = 0; i < 32; i++) {
      const float e = dt_ex2(__uint_as_float(v[i]) * (zc * 2.8853900817779268f));  // exp(2 s / softcap)
      v[i] = __float_as_uint(fmaf(-2.0f * tc, __fdividef(1.0f, e + 1.0f), tc));
    }
  } else {
#pragma unroll
    for (int i = 0; i < 32; i += 2) {
      const float2 s = make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1]));
      const float2 z = dt_mul2(s, dt_two(zc)), w = dt_mul2(z, z);
      float2 r = dt_fma2(w, dt_two(0.0010380251333117485f), dt_two(-0.0061943246982991695f));
      r = dt_fma2(r, w, dt_two(0.02027970738708973f));
      r = dt_fma2(r, w, dt_two(-0.053451646119356155f));
      r = dt_fma2(r, w, dt_two(0.13325075805187225f));
      r = dt_fma2(r, w, dt_two(-0.3333282768726349f));
      r = dt_fma2(r, w, dt_two(0.9999999403953552f));
      r = dt_mul2(r, dt_mul2(s, dt_two(uc)));
      v[i] = __float_as_uint(r.x);
      v[i + 1] = __float_as_uint(r.y);
    }
  }
}

template <int DS, int VS>
__global__ void __launch_bounds__(kDtThreads, 1)
diff_attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                    DiffTcParams p) {
  using C = DtCfg<DS, VS>;
  extern __shared__ unsigned char dt_smem_raw[];
  __shared__ __align__(8) unsigned long long q_full, full[C::SLOTS], empty[C::SLOTS], s_full[2], p_full[2], o_full;
  __shared__ uint32_t tmem_holder;
  __shared__ float xl[2][2][128], xs[4][128];  // row sums per map and half of the keys; partial sums of squares

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t smem_base = (tc_smem_u32(dt_smem_raw) + 1023u) & ~1023u;
  const uint32_t q_s = smem_base, ring = smem_base + C::Q_BYTES;
  const int head = blockIdx.x % p.heads, b = blockIdx.x / p.heads, g = head / p.group;
  const int s0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * 128;

  if (threadIdx.x == 0) {
    tc_mbar_init(tc_smem_u32(&q_full), 1);
    for (int s = 0; s < C::SLOTS; s++) {
      tc_mbar_init(tc_smem_u32(&full[s]), 1);
      tc_mbar_init(tc_smem_u32(&empty[s]), 1);
    }
    for (int m = 0; m < 2; m++) {
      tc_mbar_init(tc_smem_u32(&s_full[m]), 1);
      tc_mbar_init(tc_smem_u32(&p_full[m]), 256);
    }
    tc_mbar_init(tc_smem_u32(&o_full), 1);
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

  // key rows are indices into the [L] rows of sequence b; query token s sits at row s + L - S
  const int back = p.L - p.S;
  const long long base = p.past - back;  // token index of row 0
  const int first = p.start ? (int)max(-(1ll << 30), (long long)p.start[b] - base) : (int)max(-(1ll << 30), -base);  // row of the sequence's first token
  // first row that row r sees: the start of its chunk
  auto chunk_lo = [&](int r) -> int { return first + (r - first) / p.chunk * p.chunk; };
  const int last_r = min(p.S, s0 + 128) - 1 + back;
  const int kmin = s0 + back >= first ? chunk_lo(s0 + back) : first;
  const int j0 = max(kmin, 0) / 128;
  const int ntiles = last_r >= first ? last_r / 128 + 1 - j0 : 0;

  if (warp == 0) {
    if (lane == 0) {
      tc_mbar_expect_tx(tc_smem_u32(&q_full), C::Q_BYTES);
#pragma unroll
      for (int m = 0; m < 2; m++)
#pragma unroll
        for (int h = 0; h < DS; h++) dt_tma_3d(q_s + (m * DS + h) * C::SLAB, &tmQ, h * 64, head * 2 + m, b * p.S + s0, tc_smem_u32(&q_full));
      int slot = 0, round = 0;
      for (int it = 0; it < 3 * ntiles; it++) {
        if (round && !tc_wait(tc_smem_u32(&empty[slot]), (uint32_t)((round - 1) & 1))) { atomicExch(&g_diff_tc_err, 2u); break; }
        const int j = it / 3, what = it % 3;
        const uint32_t dst = ring + (uint32_t)slot * C::SLOT, bar = tc_smem_u32(&full[slot]);
        const int row = b * p.L + (j0 + j) * 128;
        tc_mbar_expect_tx(bar, (what < 2 ? DS : VS) * C::SLAB);
        if (what < 2) {
#pragma unroll
          for (int h = 0; h < DS; h++) dt_tma_4d(dst + h * C::SLAB, &tmK, h * 64, what, g, row, bar);
        } else {
#pragma unroll
          for (int h = 0; h < VS; h++) dt_tma_3d(dst + h * C::SLAB, &tmV, h * 64, g, row, bar);
        }
        if (++slot == C::SLOTS) { slot = 0; round++; }
      }
      // a block may end with no tile at all (padding only): the query copy must still have landed before it exits
      if (!tc_wait(tc_smem_u32(&q_full), 0)) atomicExch(&g_diff_tc_err, 9u);
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0 && ntiles > 0) {
      const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 3) << 17) | ((128u >> 4) << 24);
      const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(VS * 64 >> 3) << 17) | ((128u >> 4) << 24);
      bool ok = tc_wait(tc_smem_u32(&q_full), 0);
      if (!ok) atomicExch(&g_diff_tc_err, 3u);
      auto landed = [&](int it) -> bool { return tc_wait(tc_smem_u32(&full[it % C::SLOTS]), (uint32_t)((it / C::SLOTS) & 1)); };
      auto scores = [&](int m, int j) -> bool {
        const int it = 3 * j + m;
        if (!landed(it)) { atomicExch(&g_diff_tc_err, 4u); return false; }
        tc_fence_after();
        const uint32_t ks = ring + (uint32_t)(it % C::SLOTS) * C::SLOT, qs = q_s + m * DS * C::SLAB;
#pragma unroll
        for (int kk = 0; kk < DS * 4; kk++) {
          const uint32_t koff = (uint32_t)(kk >> 2) * C::SLAB + (uint32_t)(kk & 3) * 32;
          dt_mma_ss(tmem + C::COL_S + m * 128, tc_smem_desc(qs + koff), tc_smem_desc(ks + koff), idesc_s, kk > 0 ? 1u : 0u);
        }
        tc_commit(tc_smem_u32(&empty[it % C::SLOTS]));
        tc_commit(tc_smem_u32(&s_full[m]));
        return true;
      };
      ok = ok && scores(0, 0) && scores(1, 0);
      for (int j = 0; ok && j < ntiles; j++) {
        const int it = 3 * j + 2;
        const uint32_t vs = ring + (uint32_t)(it % C::SLOTS) * C::SLOT;
        for (int m = 0; m < 2; m++) {
          if (!tc_wait(tc_smem_u32(&p_full[m]), (uint32_t)(j & 1))) { atomicExch(&g_diff_tc_err, 5u); ok = false; break; }
          if (m == 0 && !landed(it)) { atomicExch(&g_diff_tc_err, 6u); ok = false; break; }
          tc_fence_after();
#pragma unroll
          for (int kk = 0; kk < 16; kk++) {  // 8 steps of 16 keys with the leading terms of P, then 8 with what they left out
            const uint32_t ps = tmem + C::COL_S + m * 128 + ((kk & 7) >> 1) * 32 + (kk >> 3) * 16 + (kk & 1) * 8;
            dt_mma_ts(tmem + C::COL_O + m * 128, ps, dt_desc_mn(vs + (kk & 7) * 2048, C::SLAB), idesc_o, (j > 0 || kk > 0) ? 1u : 0u);
          }
          if (m == 1) tc_commit(tc_smem_u32(&empty[it % C::SLOTS]));
          // the buffer of the next scores holds the P just issued: MMAs run in order
          if (j + 1 < ntiles && !scores(m, j + 1)) { ok = false; break; }
        }
      }
      tc_commit(tc_smem_u32(&o_full));
    }
    __syncwarp();
  } else {
    constexpr int HP = VS * 16;
    const int sub = warp & 3, m = (warp - 2) >> 3, part = ((warp - 2) >> 2) & 1;
    const uint32_t lane_base = ((uint32_t)(sub * 32)) << 16;
    const int rl = sub * 32 + lane;
    const int r = s0 + rl + back;
    const bool live = s0 + rl < p.S && r >= first;  // padding sees nothing
    const int khi = live ? r + 1 : 0, klo = live ? max(0, chunk_lo(r)) : 0;  // rows [klo, khi) are visible
    const float zc = p.scale / p.softcap, uc = p.scale * 1.4426950408889634f, tc = p.softcap * 1.4426950408889634f;
    float l_run = 0.0f;
    bool dead = false;
    for (int j = 0; j < ntiles; j++) {
      if (!tc_wait(tc_smem_u32(&s_full[m]), (uint32_t)(j & 1))) { atomicExch(&g_diff_tc_err, 8u); dead = true; break; }
      tc_fence_after();
#pragma unroll
      for (int half = 0; half < 2; half++) {
        const int gr = part * 2 + half;  // 32 keys
        const int k0 = (j0 + j) * 128 + gr * 32;
        const uint32_t col = tmem + lane_base + C::COL_S + m * 128 + gr * 32;
        uint32_t v[32];
        dt_ld_x32(col, v);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        dt_capped(v, zc, uc, tc);
        const bool plain = k0 >= klo && k0 + 32 <= khi;
        float l4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        uint32_t pk[2][16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float e0 = dt_ex2(__uint_as_float(v[i])), e1 = dt_ex2(__uint_as_float(v[i + 1]));
          if (!plain) {
            e0 = (k0 + i >= klo && k0 + i < khi) ? e0 : 0.0f;
            e1 = (k0 + i + 1 >= klo && k0 + i + 1 < khi) ? e1 : 0.0f;
          }
          l4[(i >> 1) & 3] += e0 + e1;
          const uint32_t h = dt_pack(e0, e1);
          pk[0][i >> 1] = h;
          pk[1][i >> 1] = dt_pack(e0 - __uint_as_float(h << 16), e1 - __uint_as_float(h & 0xffff0000u));
        }
        dt_st_x16(col, pk[0]);
        dt_st_x16(col + 16, pk[1]);
        l_run += (l4[0] + l4[1]) + (l4[2] + l4[3]);
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      tc_fence_before();
      tc_mbar_arrive(tc_smem_u32(&p_full[m]));
    }
    // the outputs: 128 rows, columns cut over the four warps of a quarter
    const int idx = m * 2 + part;
    xl[m][part][rl] = l_run;
    float o[HP];
#pragma unroll
    for (int i = 0; i < HP; i++) o[i] = 0.0f;
    if (ntiles > 0 && !dead && !tc_wait(tc_smem_u32(&o_full), 0)) { atomicExch(&g_diff_tc_err, 7u); dead = true; }
    asm volatile("bar.sync %0, 128;" ::"r"(1 + sub) : "memory");
    if (ntiles > 0) {
      tc_fence_after();
      const float l1 = xl[0][0][rl] + xl[0][1][rl], l2 = xl[1][0][rl] + xl[1][1][rl];
      const float i1 = l1 > 0.0f ? 1.0f / l1 : 0.0f, i2 = l2 > 0.0f ? p.lambda / l2 : 0.0f;
      uint32_t a[16], c[16];
#pragma unroll
      for (int h = 0; h < HP; h += 16) {
        tc_ld_x16(tmem + lane_base + C::COL_O + idx * HP + h, a);
        tc_ld_x16(tmem + lane_base + C::COL_O + 128 + idx * HP + h, c);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
        for (int i = 0; i < 16; i++) o[h + i] = l1 > 0.0f ? __uint_as_float(a[i]) * i1 - __uint_as_float(c[i]) * i2 : 0.0f;
      }
    }
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < HP; i++) ss = fmaf(o[i], o[i], ss);  // columns beyond vdim are zero
    xs[idx][rl] = ss;
    asm volatile("bar.sync %0, 128;" ::"r"(1 + sub) : "memory");
    ss = (xs[0][rl] + xs[1][rl]) + (xs[2][rl] + xs[3][rl]);
    const float inv = p.mult / sqrtf(ss / (float)p.vdim + p.eps);
    if (s0 + rl < p.S && !dead) {
      uint16_t* dst = p.out + ((long long)b * p.S + s0 + rl) * p.ldo + (long long)head * p.vdim + idx * HP;
#pragma unroll
      for (int i = 0; i < HP; i += 8) {
        if (idx * HP + i < p.vdim) {
          uint32_t w[4];
#pragma unroll
          for (int u = 0; u < 4; u++) w[u] = dt_pack(o[i + 2 * u] * inv, o[i + 2 * u + 1] * inv);
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

typedef CUresult (*DtEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                               const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// boxes of 128 rows (the last dimension) x 64 elements
static int dt_map(CUtensorMap* m, const void* base, int rank, const uint64_t* dims, const uint64_t* strides_elements) {
  static DtEncodeFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &ptr, 12000, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<DtEncodeFn>(ptr);
  }
  TPX_REQUIRE(fn, TPX_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
  cuuint64_t d[4], st[3];
  cuuint32_t box[4] = {64, 1, 1, 1}, es[4] = {1, 1, 1, 1};
  for (int i = 0; i < rank; i++) d[i] = dims[i];
  for (int i = 0; i + 1 < rank; i++) st[i] = strides_elements[i] * 2;
  box[rank - 1] = 128;
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(base), d, st, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  TPX_REQUIRE(r == CUDA_SUCCESS, TPX_ERR_CUDA, "diff prefill: cuTensorMapEncodeTiled failed with %d", (int)r);
  return TPX_OK;
}

template <int DS, int VS>
static int dt_launch(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const DiffTcParams& p, int64_t B, cudaStream_t st) {
  using C = DtCfg<DS, VS>;
  static bool opted[16] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 16 || !opted[dev]) {
    TPX_CUDA_OK(cudaFuncSetAttribute(diff_attn_tc_kernel<DS, VS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  TPX_CUDA_OK(launch_pdl(diff_attn_tc_kernel<DS, VS>, dim3((unsigned)(B * p.heads), (unsigned)((p.S + 127) / 128)), dim3(kDtThreads), C::SMEM, st, q, k, v, p));
  return TPX_OK;
}

bool diff_prefill_serves(int64_t dim, int64_t vdim, float softcap) {
  return dim > 0 && vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && vdim <= 128 && softcap > 0.0f && softcap <= kDiffMaxCap;
}

// The call's rows straight from proj, or from `live` (with the cached rows in reach in front of them)
int diff_prefill(const TpxDiffAttn& a, cudaStream_t st) {
  TPX_REQUIRE(a.ldp % 8 == 0 && a.ldo % 8 == 0 && a.q_col % 8 == 0 && a.k_col % 8 == 0 && a.v_col % 8 == 0, TPX_ERR_ARG, "diff prefill: bad leading dimension");
  TPX_REQUIRE((((uintptr_t)a.proj | (uintptr_t)a.live | (uintptr_t)a.out) & 15) == 0, TPX_ERR_ARG, "diff prefill: misaligned pointer");
  TPX_REQUIRE(a.B * a.heads < (1ll << 31) && a.B * a.L < (1ll << 31) && a.S <= 65535ll * 128 && a.L < (1ll << 30), TPX_ERR_UNSUPPORTED, "diff prefill: shape too large");
  const uint64_t d = (uint64_t)a.dim, e = (uint64_t)a.vdim, G = (uint64_t)a.kv_heads, R = (uint64_t)a.R, dp = (d + 15) / 16 * 16, ld = (uint64_t)a.ldp;
  const uint64_t rows = (uint64_t)(a.B * a.S), lrows = (uint64_t)(a.B * a.L);
  const uint16_t* proj = (const uint16_t*)a.proj;
  const uint16_t* live = (const uint16_t*)a.live;
  CUtensorMap mq, mk, mv;
  const uint64_t qd[3] = {d, 2 * (uint64_t)a.heads, rows}, qs[2] = {d, ld};
  const uint64_t kd[4] = {d, 2, G, lrows}, ks_p[3] = {d, 2 * d, ld}, ks_l[3] = {dp, R, G * R};
  const uint64_t vd[3] = {e, G, lrows}, vs_p[2] = {e, ld}, vs_l[2] = {R, G * R};
  int rc = dt_map(&mq, proj + a.q_col, 3, qd, qs);
  if (!rc) rc = live ? dt_map(&mk, live, 4, kd, ks_l) : dt_map(&mk, proj + a.k_col, 4, kd, ks_p);
  if (!rc) rc = live ? dt_map(&mv, live + 2 * dp, 3, vd, vs_l) : dt_map(&mv, proj + a.v_col, 3, vd, vs_p);
  if (rc) return rc;
  const DiffTcParams p = {a.start, (uint16_t*)a.out, (long long)a.ldo, (long long)a.past, (int)a.S, (int)a.L, (int)a.heads, (int)(a.heads / a.kv_heads),
                          (int)a.vdim, (int)a.chunk, a.scale, a.softcap, a.lambda, a.mult, a.eps};
  const int DS = (int)((a.dim + 63) / 64), VS = (int)((a.vdim + 63) / 64);
  switch (DS * 10 + VS) {
    case 11: return dt_launch<1, 1>(mq, mk, mv, p, a.B, st);
    case 12: return dt_launch<1, 2>(mq, mk, mv, p, a.B, st);
    case 21: return dt_launch<2, 1>(mq, mk, mv, p, a.B, st);
    default: return dt_launch<2, 2>(mq, mk, mv, p, a.B, st);
  }
}

int diff_tc_status(cudaStream_t st, unsigned* host) {
  static void* ptrs[64] = {};
  int dev = 0;
  TPX_CUDA_OK(cudaGetDevice(&dev));
  TPX_REQUIRE(dev >= 0 && dev < 64, TPX_ERR_UNSUPPORTED, "diff_status: device index %d out of range", dev);
  if (!ptrs[dev]) TPX_CUDA_OK(cudaGetSymbolAddress(&ptrs[dev], g_diff_tc_err));
  TPX_CUDA_OK(cudaMemcpyAsync(host, ptrs[dev], 4, cudaMemcpyDeviceToHost, st));
  TPX_CUDA_OK(cudaMemsetAsync(ptrs[dev], 0, 4, st));
  return TPX_OK;
}

}  // namespace tpx
