// bf16-weight linear on the 5th-generation tensor cores (tcgen05 kind::f16, sm_100a).
//
// Replaces TppBlockedLinearW<bf16> (src/csrc/fused_gemm.h:784-1073), the GEMM behind torch.ops.tpp_llm.fc_plain for
// unquantized weights; on the decoder path that is the lm_head (src/csrc/llm/fused_llm_infer.cpp:1514-1566), which the
// reference keeps in bf16 unless --quantize-lm-head is given.
//
//     y[M][N] = epilogue(x[M][K] . W[N][K]^T + bias[N])
//
// Neither operand is re-laid out: TMA reads 128-row x 64-column boxes of the plain row-major W and TOK-row boxes of x
// straight into the 128-byte-swizzled K-major operand layout; rows and columns beyond the matrices read as zero.
//
//   rows of W (output features) = M of the MMA (128 per tile), tokens = N (TOK per tile), 64 k values per k step
//   warp 0   : TMA producer into a ring of stages
//   warp 1   : allocates tensor memory, issues the MMAs (K = 16 each), commits stages back to the producer
//   warps 2-5: epilogue (tensor memory -> registers -> bias / activation / multiply / residual -> y)
//
// One CTA per SM walks a contiguous range of output tiles (the token tiles of one feature tile are neighbours, so a
// weight tile fetched for the first of them is found in L2 by the others). Up to 64 tokens the range is one of pipeline
// stages instead (BfParams::split): every CTA streams the same number of weight bytes, and the pieces of a tile that was
// cut are added in the order of k by the CTA that finishes last (fp32 partials and an arrival counter in the scratch; no
// CTA waits for another). Two accumulators in tensor memory: the
// epilogue of a tile runs under the MMAs of the next. At decode sizes the kernel is a plain stream of W at HBM rate.
#include "tpx_hybrid.cuh"
#include "tpx_tc_ptx.cuh"

namespace tpx {

// Epilogue of tpx_linear: fp32 bias, row stride, fp32 or bf16 result, activation from a column on; gated units from pairs of
// columns; or the residual sum with the norm of its next reader.
struct BfEx {
  const float *bias, *ap;
  void* y;
  long long ldy;
  int on, out_f32, act, act_from;
  uint16_t* z;
  const float *res, *add, *nw, *nb;
  float* x_out;
  uint16_t* h;
  long long ldz, ldr, ldh;
  float limit, nalpha;
};

struct BfParams {
  TcParams t;   // epilogue fields (bias, act, mul_in, res, res_scale, y, M, N, err)
  int ksteps;   // k steps of 64 (K rounded up)
  int TN, TM;   // feature tiles, token tiles
  int split;    // 1: the CTAs share all pipeline stages of all tiles evenly; a tile cut between CTAs is put together by the last of them
  BfEx ex;
};

// The stages a CTA works on, as pieces of tiles: piece = stages [g0, g1) of one tile.
struct BfPieces {
  long long u, u1;
  int ns;
  int tile, g0, g1;
  __device__ __forceinline__ BfPieces(const BfParams& p, int nstages) : ns(nstages) {
    const long long T = (long long)p.TN * p.TM;
    if (p.split) {
      const long long U = T * ns;
      u = blockIdx.x * U / gridDim.x;
      u1 = (blockIdx.x + 1) * U / gridDim.x;
    } else {
      u = blockIdx.x * T / gridDim.x * ns;
      u1 = (blockIdx.x + 1) * T / gridDim.x * ns;
    }
    tile = g0 = g1 = 0;
  }
  __device__ __forceinline__ bool next() {
    if (u >= u1) return false;
    tile = (int)(u / ns);
    g0 = (int)(u % ns);
    g1 = (int)min((long long)ns, g0 + (u1 - u));
    u += g1 - g0;
    return true;
  }
};

// 16 consecutive tokens of output feature n; the lanes of a warp hold 32 neighbouring features
__device__ __forceinline__ void bf_finish16_ex(const BfEx& e, int M, int tok0, int n, const float (&v)[16]) {
  const int live = M - tok0;
  const float b = e.bias ? e.bias[n] : 0.0f;
  float x[16];
#pragma unroll
  for (int j = 0; j < 16; j++) x[j] = v[j] + b;
  if (e.x_out) {
    const float add = e.add ? e.add[n] : 0.0f, w = e.nw[n], nb = e.nb[n];
    const float* r = e.res + (long long)tok0 * e.ldr + n;
    float* xo = e.x_out + (long long)tok0 * e.ldr + n;
    uint16_t* h = e.h + (long long)tok0 * e.ldh + n;
    float s[16];
#pragma unroll
    for (int j = 0; j < 16; j++) s[j] = j < live ? __ldcs(r + j * e.ldr) : 0.0f;
#pragma unroll
    for (int j = 0; j < 16; j++) {
      s[j] += x[j] + add;
      if (j < live) xo[j * e.ldr] = s[j];
    }
#pragma unroll
    for (int j = 0; j < 16; j++)
      if (j < live) h[j * e.ldh] = f32_to_bf16_bits(fmaf(tanhf(e.nalpha * s[j]), w, nb));
    return;
  }
  if (e.act && n >= e.act_from) {
    const float a0 = e.ap ? e.ap[0] : 0.0f, a1 = e.ap ? e.ap[1] : 0.0f;
#pragma unroll
    for (int j = 0; j < 16; j++) x[j] = hy_act(x[j], e.act, a0, a1);
  }
  if (e.out_f32) {
    float* y = reinterpret_cast<float*>(e.y) + (long long)tok0 * e.ldy + n;
#pragma unroll
    for (int j = 0; j < 16; j++)
      if (j < live) y[j * e.ldy] = x[j];
  } else {
    uint16_t* y = reinterpret_cast<uint16_t*>(e.y) + (long long)tok0 * e.ldy + n;
#pragma unroll
    for (int j = 0; j < 16; j++)
      if (j < live) y[j * e.ldy] = f32_to_bf16_bits(x[j]);
  }
}

// The same where the features are pairs (g, u) of neighbouring lanes: the lane of g finishes the first eight tokens, the lane
// of u the others. Called by whole warps; lanes with n < act_from take part in the exchange only.
__device__ __forceinline__ void bf_finish16_glu(const BfEx& e, int M, int N, int tok0, int n, const float (&v)[16]) {
  const int live = M - tok0, up = n & 1;
  const float b = (e.bias && n < N) ? e.bias[n] : 0.0f;
  uint16_t* z = e.z + (long long)(tok0 + up * 8) * e.ldz + (n - e.act_from) / 2;
#pragma unroll
  for (int j = 0; j < 8; j++) {
    const float lo = v[j] + b, hi = v[j + 8] + b;
    const float other = __shfl_xor_sync(0xffffffffu, up ? lo : hi, 1);
    const float r = hy_clamped_glu_fast(up ? other : lo, up ? hi : other, e.limit);
    if (n >= e.act_from && n < N && up * 8 + j < live) z[j * e.ldz] = f32_to_bf16_bits(r);
  }
}

template <int TOK>
struct BfCfg {
  static constexpr int UK = TOK <= 64 ? 2 : 1;           // k steps per pipeline stage
  static constexpr int A_BYTES = 128 * 128;              // 128 features x 64 bf16
  static constexpr int B_BYTES = TOK * 128;              // TOK tokens x 64 bf16
  static constexpr int STAGE_BYTES = UK * (A_BYTES + B_BYTES);
  static constexpr int STAGES_FIT = (227 * 1024 - 3072) / STAGE_BYTES;
  static constexpr int STAGES = STAGES_FIT > 10 ? 10 : STAGES_FIT;
  static constexpr int COLS_RAW = 2 * TOK;               // two accumulators
  static constexpr int TMEM_COLS = COLS_RAW <= 32 ? 32 : COLS_RAW <= 64 ? 64 : COLS_RAW <= 128 ? 128 : COLS_RAW <= 256 ? 256 : 512;
  static constexpr size_t SMEM = (size_t)STAGES * STAGE_BYTES + 1024;
  static_assert(STAGES >= 3, "at least three stages");
  static_assert(COLS_RAW <= 512, "tensor memory");
};

__device__ __forceinline__ void bf_mma(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{ .reg .pred p; setp.ne.b32 p, %4, 0;\n"
      "  tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }" ::"r"(d_tmem),
      "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}

template <int TOK>
__global__ void __launch_bounds__(kTcThreads, 1)
linear_bf16_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmX, BfParams p) {
  using C = BfCfg<TOK>;
  extern __shared__ unsigned char bf_smem_raw[];
  __shared__ __align__(8) unsigned long long bar_full[C::STAGES], bar_empty[C::STAGES];
  __shared__ __align__(8) unsigned long long acc_full[2], acc_empty[2];
  __shared__ uint32_t tmem_holder;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t smem_base = (tc_smem_u32(bf_smem_raw) + 1023u) & ~1023u;
  const int nstages = (p.ksteps + C::UK - 1) / C::UK;  // pipeline stages per tile
  __shared__ int last_piece;

  if (threadIdx.x == 0) {
    for (int s = 0; s < C::STAGES; s++) {
      tc_mbar_init(tc_smem_u32(&bar_full[s]), 1);
      tc_mbar_init(tc_smem_u32(&bar_empty[s]), 1);
    }
    for (int b = 0; b < 2; b++) {
      tc_mbar_init(tc_smem_u32(&acc_full[b]), 1);
      tc_mbar_init(tc_smem_u32(&acc_empty[b]), 4);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tc_smem_u32(&tmem_holder)),
                 "r"((uint32_t)C::TMEM_COLS)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_holder;
  pdl_trigger();

  if (warp == 0) {
    // ------------------------------------------------------------ producer
    if (lane == 0) {
      // at decode sizes W is a model's weight, not the output of a kernel in flight: its copies for the first stages need not
      // wait for the kernels that make x (many rows may come with a weight unpacked for the call)
      auto copy_w = [&](int tile, int g, int s) {
        const uint32_t st = smem_base + (uint32_t)s * C::STAGE_BYTES;
        const uint32_t bar = tc_smem_u32(&bar_full[s]);
        tc_mbar_expect_tx(bar, C::STAGE_BYTES);
#pragma unroll
        for (int u = 0; u < C::UK; u++)  // a k step beyond K reads as zeros
          tc_tma_2d(st + u * C::A_BYTES, &tmW, (g * C::UK + u) * 64, tile / p.TM * 128, bar);
      };
      auto copy_x = [&](int tile, int g, int s) {
        const uint32_t st = smem_base + (uint32_t)s * C::STAGE_BYTES;
        const uint32_t bar = tc_smem_u32(&bar_full[s]);
#pragma unroll
        for (int u = 0; u < C::UK; u++)
          tc_tma_2d(st + C::UK * C::A_BYTES + u * C::B_BYTES, &tmX, (g * C::UK + u) * 64, tile % p.TM * TOK, bar);
      };
      BfPieces ahead(p, nstages);
      int pre = 0;
      while (TOK <= 64 && pre < C::STAGES && ahead.next())
        for (int g = ahead.g0; g < ahead.g1 && pre < C::STAGES; g++) copy_w(ahead.tile, g, pre++);
      pdl_wait();
      BfPieces pc(p, nstages);
      long long it = 0;
      bool dead = false;
      while (!dead && pc.next()) {
        for (int g = pc.g0; g < pc.g1; g++, it++) {
          const int s = (int)(it % C::STAGES);
          if (it >= C::STAGES && !tc_wait(tc_smem_u32(&bar_empty[s]), (uint32_t)((it / C::STAGES - 1) & 1))) {
            atomicExch(p.t.err, 2u);
            dead = true;
            break;
          }
          if (it >= pre) copy_w(pc.tile, g, s);
          copy_x(pc.tile, g, s);
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      // kind::f16: D = F32 (1), A = B = BF16 (1), both K-major, N = TOK, M = 128
      const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TOK >> 3) << 17) | ((128u >> 4) << 24);
      long long it = 0;
      uint32_t empty_phase = 0;  // bit b: parity to wait for on acc_empty[b]
      bool dead = false;
      BfPieces pc(p, nstages);
      for (int i = 0; !dead && pc.next(); i++) {
        const int buf = i & 1;
        if (i >= 2) {  // the epilogue must have drained this accumulator
          if (!tc_wait(tc_smem_u32(&acc_empty[buf]), (empty_phase >> buf) & 1u)) { atomicExch(p.t.err, 3u); break; }
          empty_phase ^= 1u << buf;
          tc_fence_after();
        }
        for (int g = pc.g0; g < pc.g1; g++, it++) {
          const int s = (int)(it % C::STAGES);
          if (!tc_wait(tc_smem_u32(&bar_full[s]), (uint32_t)((it / C::STAGES) & 1))) { atomicExch(p.t.err, 4u); dead = true; break; }
          tc_fence_after();
          const uint32_t st = smem_base + (uint32_t)s * C::STAGE_BYTES;
#pragma unroll
          for (int u = 0; u < C::UK; u++) {
#pragma unroll
            for (int j = 0; j < 4; j++) {
              bf_mma(tmem + buf * TOK, tc_smem_desc(st + u * C::A_BYTES) + (uint64_t)(2 * j),
                     tc_smem_desc(st + C::UK * C::A_BYTES + u * C::B_BYTES) + (uint64_t)(2 * j), idesc, (g == pc.g0 && u == 0 && j == 0) ? 0u : 1u);
            }
          }
          tc_commit(tc_smem_u32(&bar_empty[s]));
        }
        if (!dead) tc_commit(tc_smem_u32(&acc_full[buf]));
      }
    }
    __syncwarp();
  } else {
    // ------------------------------------------------------------ epilogue (warps 2..5)
    const int sub = warp & 3;  // tensor-memory lanes 32*sub .. 32*sub+31 belong to this warp
    const uint32_t lane_base = ((uint32_t)(sub * 32)) << 16;
    uint32_t full_phase = 0;
    pdl_wait();  // residual and multiplier inputs belong to earlier grids
    BfPieces pc(p, nstages);
    const int first_tile = (int)(pc.u / nstages);
    bool dead = false;  // a warp that gave up still meets the others at their barriers
    for (int i = 0; pc.next(); i++) {
      const int buf = i & 1;
      if (!dead && !tc_wait(tc_smem_u32(&acc_full[buf]), (full_phase >> buf) & 1u)) {
        if (lane == 0) atomicExch(p.t.err, 6u);
        dead = true;
      }
      full_phase ^= 1u << buf;
      tc_fence_after();
      const int tn = pc.tile / p.TM, tm = pc.tile % p.TM;
      const int nl = sub * 32 + lane, n = tn * 128 + nl;
      const int tok0 = tm * TOK;
      const bool whole = pc.g0 == 0 && pc.g1 == nstages;
      float* part = whole ? nullptr : p.t.partial + ((size_t)blockIdx.x * 2 + (pc.tile == first_tile ? 0 : 1)) * TOK * 128;
      const bool pairs = p.ex.on && p.ex.act == TPX_ACT_CLAMPED_GLU && tn * 128 + sub * 32 + 31 >= p.ex.act_from;  // per warp
      auto finish = [&](int c0, const float (&v)[16]) {
        if (pairs) {
          if (tok0 + c0 >= p.t.M) return;
          bf_finish16_glu(p.ex, p.t.M, p.t.N, tok0 + c0, n, v);
          if (n >= p.ex.act_from) return;
        }
        if (n < p.t.N && tok0 + c0 < p.t.M) {
          const float v2[16] = {};
          if (p.ex.on) bf_finish16_ex(p.ex, p.t.M, tok0 + c0, n, v);
          else tc_finish16<false>(p.t, tok0 + c0, n, v, v2);
        }
      };
#pragma unroll 1
      for (int c0 = 0; c0 < TOK && !dead; c0 += 16) {
        uint32_t a[16];
        float v[16];
        tc_ld_x16(tmem + lane_base + buf * TOK + c0, a);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
        for (int j = 0; j < 16; j++) v[j] = __uint_as_float(a[j]);
        if (whole) finish(c0, v);
        else if (tok0 + c0 < p.t.M) {
#pragma unroll
          for (int j = 0; j < 16; j++) part[(c0 + j) * 128 + nl] = v[j];
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) tc_mbar_arrive(tc_smem_u32(&acc_empty[buf]));
      if (!whole) {
        // publish this piece; whoever comes last adds the tile's pieces in the order of k
        const long long U = (long long)p.TN * p.TM * nstages, G = gridDim.x, u = (long long)pc.tile * nstages;
        const int ca = (int)(((u + 1) * G - 1) / U), cb = (int)(((u + nstages) * G - 1) / U);
        __threadfence();
        asm volatile("bar.sync 1, 128;" ::: "memory");
        if (threadIdx.x == 64) {
          const bool last = atomicAdd(p.t.counters + pc.tile, 1u) == (unsigned)(cb - ca);
          if (last) p.t.counters[pc.tile] = 0;
          last_piece = last;
        }
        asm volatile("bar.sync 1, 128;" ::: "memory");
        if (last_piece) {
          __threadfence();
#pragma unroll 1
          for (int c0 = 0; c0 < TOK && tok0 + c0 < p.t.M; c0 += 16) {
            float v[16] = {};
            for (int c = ca; c <= cb; c++) {
              const float* q = p.t.partial + ((size_t)c * 2 + ((int)(c * U / G / nstages) == pc.tile ? 0 : 1)) * TOK * 128 + c0 * 128 + nl;
#pragma unroll
              for (int j = 0; j < 16; j++) v[j] += __ldcg(q + j * 128);
            }
            finish(c0, v);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((uint32_t)C::TMEM_COLS) : "memory");
  }
}

// 2-D bf16 tensor [rows][cols] (row stride ld elements), box = 64 columns x box_rows, 128-byte swizzle.
static int bf_make_map(CUtensorMap* m, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows) {
  typedef CUresult (*Fn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                         const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
  static Fn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &ptr, 12000, cudaEnableDefault, &q) == cudaSuccess &&
        q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<Fn>(ptr);
  }
  TPX_REQUIRE(fn, TPX_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
  cuuint64_t gdim[2] = {cols, rows};
  cuuint64_t gstr[1] = {ld * 2};
  cuuint32_t box[2] = {64, box_rows};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), gdim, gstr, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  TPX_REQUIRE(r == CUDA_SUCCESS, TPX_ERR_CUDA, "cuTensorMapEncodeTiled failed with %d (rows=%llu cols=%llu box_rows=%u)", (int)r,
              (unsigned long long)rows, (unsigned long long)cols, box_rows);
  return TPX_OK;
}

template <int TOK>
static int bf_launch(const CUtensorMap& w, const CUtensorMap& x, const BfParams& p, cudaStream_t st) {
  using C = BfCfg<TOK>;
  static bool opted[16] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 16 || !opted[dev]) {
    TPX_CUDA_OK(cudaFuncSetAttribute(linear_bf16_kernel<TOK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    if (dev >= 0 && dev < 16) opted[dev] = true;
  }
  const long long T = (long long)p.TN * p.TM;
  const int sms = sm_count();
  const int grid = p.split ? p.split : (int)(T < sms ? T : sms);
  TPX_CUDA_OK(launch_pdl(linear_bf16_kernel<TOK>, dim3((unsigned)grid), dim3(kTcThreads), C::SMEM, st, w, x, p));
  return TPX_OK;
}

// Decode sizes read every weight once: with whole tiles per CTA the rate is set by the CTA that has one tile more than the
// others, or by the few CTAs that have any. CTAs of an even split of all stages (0: keep whole tiles).
static int bf_split_ctas(int64_t M, int64_t N, int64_t K) {
  if (M > 64) return 0;
  const int64_t T = (N + 127) / 128, ns = ((K + 63) / 64 + 1) / 2, sms = sm_count();
  if (T >= 8 * sms || T % sms == 0 || T > 16000) return 0;
  const int64_t most = T * ns / 4;  // a CTA takes at least four stages (512 values of k)
  const int64_t grid = most < sms ? most : sms;
  return grid > T || T > sms ? (int)grid : 0;
}
static size_t bf_split_bytes(int64_t M, int grid) { return (size_t)grid * 2 * (M <= 16 ? 16 : M <= 32 ? 32 : 64) * 128 * 4; }

// Tiles, tensor maps and launch for a filled epilogue.
static int bf_run(BfParams& p, const void* w, const void* x, int64_t M, int64_t N, int64_t K, int64_t ldw, int64_t ldx, void* scratch,
                  size_t scratch_bytes, cudaStream_t st) {
  p.split = bf_split_ctas(M, N, K);
  if (p.split && scratch_bytes < kTcCounterBytes + bf_split_bytes(M, p.split)) p.split = 0;
  p.t.counters = reinterpret_cast<unsigned*>(scratch);
  p.t.partial = reinterpret_cast<float*>(reinterpret_cast<unsigned char*>(scratch) + kTcCounterBytes);
  const int tok = M <= 16 ? 16 : M <= 32 ? 32 : M <= 64 ? 64 : M <= 128 ? 128 : 256;
  p.t.M = (int)M; p.t.N = (int)N; p.t.K = (int)K;
  p.ksteps = (int)((K + 63) / 64);
  p.TN = (int)((N + 127) / 128);
  p.TM = (int)((M + tok - 1) / tok);
  CUtensorMap mw, mx;
  int rc = bf_make_map(&mw, w, (uint64_t)N, (uint64_t)K, (uint64_t)ldw, 128);
  if (rc) return rc;
  rc = bf_make_map(&mx, x, (uint64_t)M, (uint64_t)K, (uint64_t)ldx, (uint32_t)tok);
  if (rc) return rc;
  switch (tok) {
    case 16: return bf_launch<16>(mw, mx, p, st);
    case 32: return bf_launch<32>(mw, mx, p, st);
    case 64: return bf_launch<64>(mw, mx, p, st);
    case 128: return bf_launch<128>(mw, mx, p, st);
    default: return bf_launch<256>(mw, mx, p, st);
  }
}

int linear_tc_ex(const TpxLinear& a, cudaStream_t st) {
  TPX_REQUIRE(a.K % 8 == 0 && a.ldx % 8 == 0 && a.ldw % 8 == 0, TPX_ERR_ARG, "linear: bf16 rows must be whole 16-byte units (K=%ld ldx=%ld ldw=%ld)",
              (long)a.K, (long)a.ldx, (long)a.ldw);
  TPX_REQUIRE((((uintptr_t)a.w | (uintptr_t)a.x) & 15) == 0 && ((uintptr_t)a.scratch & 255) == 0, TPX_ERR_ARG, "linear: misaligned pointer");
  TPX_REQUIRE(a.scratch && a.scratch_bytes >= kTcCounterBytes, TPX_ERR_SCRATCH, "linear: scratch of %zu bytes needed, %zu given", kTcCounterBytes,
              a.scratch_bytes);
  BfParams p = {};
  p.t.err = reinterpret_cast<unsigned*>(reinterpret_cast<unsigned char*>(a.scratch) + kTcCounterBytes - 4);
  p.ex = {a.bias, a.act_params, a.y, (long long)a.ldy, 1, a.out_f32, a.act, a.act_from, (uint16_t*)a.z, a.res, a.add, a.norm_w, a.norm_b, a.x_out,
          (uint16_t*)a.h, (long long)a.ldz, (long long)a.ldr, (long long)a.ldh, a.limit, a.norm_alpha};
  return bf_run(p, a.w, a.x, a.M, a.N, a.K, a.ldw, a.ldx, a.scratch, a.scratch_bytes, st);
}

}  // namespace tpx

using namespace tpx;

extern "C" size_t tpx_linear_bf16_tc_scratch_bytes(int64_t M, int64_t N, int64_t K) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  const int grid = bf_split_ctas(M, N, K);
  return kTcCounterBytes + (grid ? bf_split_bytes(M, grid) : 0);
}

extern "C" int tpx_linear_bf16_tc(const uint16_t* w, const uint16_t* x, int64_t M, int64_t N, int64_t K, const uint16_t* bias, int act,
                                  const uint16_t* mul_in, const uint16_t* res, float res_scale, uint16_t* y, void* scratch,
                                  size_t scratch_bytes, void* stream) {
  TPX_REQUIRE(M >= 0 && N > 0 && K > 0, TPX_ERR_ARG, "linear_bf16_tc: bad shape");
  if (M == 0) return TPX_OK;
  TPX_REQUIRE(w && x && y, TPX_ERR_ARG, "linear_bf16_tc: null pointer");
  TPX_REQUIRE(K % 8 == 0, TPX_ERR_ARG, "linear_bf16_tc: K must be a multiple of 8 (rows of whole 16-byte units), got %ld", (long)K);
  TPX_REQUIRE(M < (1 << 24) && N < (1 << 24) && K < (1 << 24), TPX_ERR_ARG, "linear_bf16_tc: shape too large");
  TPX_REQUIRE(act >= TPX_ACT_NONE && act <= TPX_ACT_RELU, TPX_ERR_ARG, "linear_bf16_tc: unknown activation %d", act);
  TPX_REQUIRE((((uintptr_t)w | (uintptr_t)x) & 15) == 0 && ((uintptr_t)scratch & 255) == 0, TPX_ERR_ARG, "linear_bf16_tc: misaligned pointer");
  TPX_REQUIRE(scratch && scratch_bytes >= kTcCounterBytes, TPX_ERR_SCRATCH, "linear_bf16_tc: scratch of %zu bytes needed, %zu given",
              kTcCounterBytes, scratch_bytes);
  BfParams p = {};
  p.t.bias = bias; p.t.mul_in = mul_in; p.t.res = res; p.t.res_scale = res_scale; p.t.y = y; p.t.act = act;
  p.t.err = reinterpret_cast<unsigned*>(reinterpret_cast<unsigned char*>(scratch) + kTcCounterBytes - 4);
  return bf_run(p, w, x, M, N, K, K, K, scratch, scratch_bytes, (cudaStream_t)stream);
}
