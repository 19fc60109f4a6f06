// Host-side pieces that every library of this package contains: error text, launch check, the launch-overlap switch.
#include <cstdarg>
#include <cstdio>
#include <cstdlib>

#include "common.cuh"

namespace b200 {

static thread_local char g_err[512] = "";

void set_error(const char* fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(g_err, sizeof(g_err), fmt, ap);
  va_end(ap);
}

bool pdl_enabled() {
  static const int on = [] {
    const char* v = getenv("B200_PDL");
    return (v != nullptr && v[0] == '0') ? 0 : 1;
  }();
  return on != 0;
}

int check_launch(const char* what) {
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) {
    set_error("%s: %s", what, cudaGetErrorString(e));
    return B200_E_CUDA;
  }
  return B200_OK;
}

}  // namespace b200

extern "C" const char* b200_last_error_string(void) { return b200::g_err; }
