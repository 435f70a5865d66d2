// C-ABI entry points that are not tied to one kernel file: error text, device info, kernel-selection switches.
#include "tpx_common.cuh"
#include <string.h>
#include <stdlib.h>

namespace tpx {

static thread_local char g_err[512] = "";

void set_error(const char* fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(g_err, sizeof(g_err), fmt, ap);
  va_end(ap);
}

static unsigned long long g_launches = 0;  // relaxed tally; exact when one host thread launches
void count_launch() { __atomic_fetch_add(&g_launches, 1ull, __ATOMIC_RELAXED); }

static Knobs g_knobs;
static bool g_knobs_read = false;

static void read_knobs() {
  auto env = [](const char* name, int dflt) { const char* e = getenv(name); return e ? atoi(e) : dflt; };
  g_knobs.tc_whole = env("TPX_TC_WHOLE", -1);
  g_knobs.tc_wide = env("TPX_TC_WIDE", -1);
  g_knobs.tc_f4 = env("TPX_TC_F4", -1);
  g_knobs.tc_w4 = env("TPX_TC_W4", -1);
  g_knobs.tc4_occ = env("TPX_TC4_OCC", 1);
  g_knobs.tc_cluster = env("TPX_TC_CLUSTER", 1);
  g_knobs.tc_pf = env("TPX_TC_PF", 0);
  g_knobs.handoff_min = env("TPX_HANDOFF_MIN_TOKENS", 33);
  g_knobs.tc_p = env("TPX_TC_P", -1);
  g_knobs.tc_p2 = env("TPX_TC_P2", -1);
  g_knobs.tc_p_rows = env("TPX_TC_P_ROWS", 1);
  g_knobs.tc_p_uks = env("TPX_TC_P_UKS", 2);
  g_knobs.attn_splits = env("TPX_ATTN_SPLITS", 0);
  g_knobs.attn_tc = env("TPX_ATTN_TC", 1);
  g_knobs.pdl = env("TPX_PDL", 1) != 0;
#ifdef TPX_DEBUG
  g_knobs.dbg = env("TPX_TC_DBG", 0);
#else
  g_knobs.dbg = 0;
#endif
  g_knobs_read = true;
}

const Knobs& knobs() {
  if (!g_knobs_read) read_knobs();
  return g_knobs;
}

int sm_count() {
  static int cached[64] = {0};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 148;
  if (cached[dev] == 0) {
    int n = 0;
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
    cached[dev] = n;
  }
  return cached[dev];
}

__global__ void e2m1_pair_table_kernel(uint32_t* out) {
  uint32_t b = threadIdx.x;
  uint32_t r;
  asm("{ .reg .b8 t; cvt.u8.u32 t, %1; cvt.rn.f16x2.e2m1x2 %0, t; }" : "=r"(r) : "r"(b));
  out[b] = r;
}

}  // namespace tpx

using namespace tpx;

extern "C" int tpx_version(void) { return 100; }
extern "C" const char* tpx_last_error(void) { return g_err; }
extern "C" int tpx_sm_count(void) { return sm_count(); }
extern "C" void tpx_reload_options(void) { read_knobs(); }

extern "C" int tpx_e2m1_pair_table(uint32_t* out256, void* stream) {
  TPX_REQUIRE(out256, TPX_ERR_ARG, "e2m1_pair_table: null pointer");
  e2m1_pair_table_kernel<<<1, 256, 0, (cudaStream_t)stream>>>(out256);
  TPX_LAUNCH_OK();
  return TPX_OK;
}

extern "C" unsigned long long tpx_launch_count(void) { return __atomic_load_n(&tpx::g_launches, __ATOMIC_RELAXED); }
