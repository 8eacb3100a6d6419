/* absent_parallel.cu -- stands for what only Llama decoders and decoders of parallel
 * blocks use, in the library that leaves them out. */
#include "absent.h"

namespace vxb {

ABSENT(rowdot_f32, int, RowDotParams &, Stream)
ABSENT(rowdot_bf16, int, RowDotParams &, Stream)
int rowdot_f32_status() { return 0; }
int rowdot_bf16_status() { return 0; }

} // namespace vxb

void decoder_record_parallel_step(vx_decoder *) {}
void decoder_free_parallel(vx_decoder *) {}
void decoder_parallel_rows(vx_decoder *, const int32_t *, int, const int32_t *, int,
                           float *) {}

extern "C" vx_decoder *vx_decoder_create_parallel(const vx_parallel_config *) {
  vxb::set_last_error(NOT_HERE("vx_decoder_create_parallel"));
  return nullptr;
}
