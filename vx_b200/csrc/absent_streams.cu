/* absent_streams.cu -- stands for what only decoders of several residual streams use,
 * in the library that leaves them out. */
#include "absent.h"

namespace vxb {

ABSENT(rowdot_streams_f32, int, RowDotParams &, Stream)
ABSENT(rowdot_streams_bf16, int, RowDotParams &, Stream)
int latent_status() { return 0; }
int gated_linear_status() { return 0; }
int rowdot_streams_f32_status() { return 0; }
int rowdot_streams_bf16_status() { return 0; }

} // namespace vxb

void decoder_record_stream_step(vx_decoder *) {}
void decoder_free_streams(vx_decoder *) {}
void decoder_stream_rows(vx_decoder *, const int32_t *, int, const int32_t *, int, float *) {}

extern "C" vx_decoder *vx_decoder_create_streams(const vx_stream_config *) {
  vxb::set_last_error(NOT_HERE("vx_decoder_create_streams"));
  return nullptr;
}
