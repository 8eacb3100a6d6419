/* absent.cu -- the launchers that the libraries for one kind of decoder leave out
 * (vx_b200/build.py): each refuses, and the status words are 0.  The whole library has
 * the kernels themselves in their place.  absent_parallel.cu and absent_streams.cu
 * stand for the other kind of decoder. */
#include "absent.h"

namespace vxb {

ABSENT(gemm_f32, const float *, int64_t, const float *, int64_t, float *, int64_t, int64_t,
       int64_t, int64_t, Stream)
ABSENT(gemm_f32_split, const float *, int64_t, const float *, int64_t, float *, int64_t,
       int64_t, int64_t, int64_t, void *, Stream)
ABSENT(gemm_f64, const double *, int64_t, const double *, int64_t, double *, int64_t,
       int64_t, int64_t, int64_t, Stream)
ABSENT(gemm_16, bool, const void *, int64_t, const void *, int64_t, void *, int64_t,
       int64_t, int64_t, int64_t, Stream)
ABSENT(gemm_16_route, int, bool, const void *, int64_t, const void *, int64_t, void *,
       int64_t, int64_t, int64_t, int64_t, void *, Stream)
ABSENT(batched_proj, const BatchedProj &, Stream)
ABSENT(decode_step, const StepArgs &, Stream)
ABSENT(flash_attention_fwd, const void *, const void *, const void *, void *, int, int,
       int, int, float, bool, Stream)
ABSENT(rowdot_quant, int, RowDotParams &, int, Stream)
ABSENT(rows_gemm_q4, const void *, const void *, const void *, int, int, int, float *,
       Stream)
ABSENT(rows_gemm_fp8, const void *, const void *, const void *, int, int, int, float *,
       Stream)
ABSENT(gemm_q4, float *, const void *, const void *, const float *, int, int, int, Stream)
ABSENT(gemm_fp8, float *, const void *, const void *, const float *, int, int, int, Stream)
ABSENT(moe_group_count, int32_t *, int64_t, const int32_t *, int, int, Stream)
ABSENT(moe_group_offsets, int32_t *, int64_t, int32_t *, int32_t *, int, int32_t *, int,
       const int32_t *, int64_t, int, int, int, Stream)
ABSENT(moe_group_place, int32_t *, int, const int32_t *, const int32_t *, int64_t, int,
       int, Stream)
ABSENT(moe_swiglu_q4_grouped, const MoeGroupedArgs &, Stream)
ABSENT(moe_down_q4_add_grouped, const MoeGroupedArgs &, Stream)
ABSENT(fill_normal, void *, bool, int64_t, uint64_t, float, Stream)
ABSENT(fill_uniform, void *, bool, int64_t, uint64_t, float, float, Stream)
ABSENT(quantize_fp8, const void *, int, int, void *, float *, Stream)
ABSENT(quantize_q4, const void *, int, int, void *, void *, Stream)
ABSENT(interleave_gathered, const void *, void *, int, int64_t, int64_t, int, Stream)

size_t gemm_f32_split_scratch_bytes(int64_t, int64_t, int64_t, int64_t) { return 0; }
size_t batched_proj_scratch_floats(int, int) { return 0; }
size_t step_scratch_floats(int) { return 0; }
int gemm_status(Stream) { return 0; }
int flash_status(Stream) { return 0; }
int step_status(Stream) { return 0; }
int batched_proj_status(Stream) { return 0; }
int moe_group_status(Stream) { return 0; }
int rowdot_quant_status() { return 0; }

} // namespace vxb

extern "C" int32_t vx_b200_attention_decode_static(float *, const float *, const float *,
                                                   const float *, int32_t, int32_t,
                                                   int32_t, int32_t) {
  vxb::set_last_error(NOT_HERE("vx_b200_attention_decode_static"));
  return -1;
}
