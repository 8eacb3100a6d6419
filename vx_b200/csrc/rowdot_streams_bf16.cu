/* rowdot_streams_bf16.cu -- the projection kernel with bf16 weights around a residual
 * of several streams: their weighted sum and its norm in front, or their mixing
 * behind. */
#include "rowdot.cuh"

namespace vxb {

const char *rowdot_streams_bf16(int epi, RowDotParams &p, cudaStream_t stream) {
  switch (epi) {
  case EPI_IN_STORE: return launch_rowdot_w<__nv_bfloat16, EPI_IN_STORE>(p, stream);
  case EPI_IN_GELU: return launch_rowdot_w<__nv_bfloat16, EPI_IN_GELU>(p, stream);
  case EPI_IN_LOGITS: return launch_rowdot_w<__nv_bfloat16, EPI_IN_LOGITS>(p, stream);
  case EPI_MIX: return launch_rowdot_w<__nv_bfloat16, EPI_MIX>(p, stream);
  default: return "unknown epilogue";
  }
}

int rowdot_streams_bf16_status() { return take_rowdot_status(); }

} // namespace vxb
