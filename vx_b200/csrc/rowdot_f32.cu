/* rowdot_f32.cu -- the projection kernel with f32 weights, every epilogue. */
#include "rowdot.cuh"

namespace vxb {

const char *rowdot_f32(int epi, RowDotParams &p, cudaStream_t stream) {
  switch (epi) {
  case EPI_STORE: return launch_rowdot_w<float, EPI_STORE>(p, stream);
  case EPI_ADD: return launch_rowdot_w<float, EPI_ADD>(p, stream);
  case EPI_BIAS: return launch_rowdot_w<float, EPI_BIAS>(p, stream);
  case EPI_SWIGLU: return launch_rowdot_w<float, EPI_SWIGLU>(p, stream);
  case EPI_QKV: return launch_rowdot_w<float, EPI_QKV>(p, stream);
  case EPI_PUSH: return launch_rowdot_w<float, EPI_PUSH>(p, stream);
  case EPI_FAN: return launch_rowdot_w<float, EPI_FAN>(p, stream);
  default: return "unknown epilogue";
  }
}

int rowdot_f32_status() { return take_rowdot_status(); }

} // namespace vxb
