/* launch_util.h -- what every launcher asks of the runtime. */
#ifndef VXB_LAUNCH_UTIL_H
#define VXB_LAUNCH_UTIL_H

#include <cuda_runtime.h>

#include <cstdio>

namespace vxb {
namespace {

[[maybe_unused]] int sm_count() {
  static int n = [] {
    int dev = 0, v = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev);
    return v > 0 ? v : 148;
  }();
  return n;
}

[[maybe_unused]] const char *check_launch(const char *what) {
  const cudaError_t e = cudaGetLastError();
  if (e == cudaSuccess)
    return nullptr;
  static thread_local char msg[256];
  snprintf(msg, sizeof msg, "%s: %s", what, cudaGetErrorString(e));
  return msg;
}

} // namespace
} // namespace vxb

#endif /* VXB_LAUNCH_UTIL_H */
