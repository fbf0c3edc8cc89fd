// Host-side helpers of a C-ABI translation unit: error text, argument checks, launches with programmatic
// stream serialisation, the count of launches.  Everything is local to the including unit.
#pragma once

#include <cuda_runtime.h>

#include <cstdio>
#include <cstdlib>
#include <string>
#include <utility>

namespace {

thread_local std::string g_last_error;
long long g_launches = 0;

int fail(int code, const char* fmt, const char* detail = "") {
  char buf[512];
  snprintf(buf, sizeof(buf), fmt, detail);
  g_last_error = buf;
  return code;
}
#define TB_CUDA(expr)                                                        \
  do {                                                                       \
    cudaError_t e__ = (expr);                                                \
    if (e__ != cudaSuccess) return fail(TB_ECUDA, #expr ": %s", cudaGetErrorString(e__)); \
  } while (0)
#define TB_REQUIRE(cond) \
  do {                   \
    if (!(cond)) return fail(TB_EINVAL, "requirement failed: %s", #cond); \
  } while (0)

// Every kernel is launched with programmatic stream serialisation (see pdl_wait in common.cuh);
// TILERT_B200_PDL=0 in the environment switches it off.
bool pdl_enabled() {
  static const bool on = [] {
    const char* e = getenv("TILERT_B200_PDL");
    return e == nullptr || e[0] != '0';
  }();
  return on;
}
template <typename... KArgs, typename... Args>
cudaError_t launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}

}  // namespace
