/* rowdot_quant.cu -- the projections with fp8 and Q4_0 weights: on the tensor
 * cores where the shape allows (rowdot_quant_mma.cuh), else on the FMA pipe. */
#include "rowdot.cuh"

namespace vxb {
namespace {

#include "rowdot_quant_mma.cuh"

template <int EPI>
const char *either_format(RowDotParams &p, int fmt, cudaStream_t stream) {
  const char *r = fmt == kFmtFp8 ? launch_quant_mma<Fp8W, EPI>(p, stream)
                                 : launch_quant_mma<Q4W, EPI>(p, stream);
  if (!r || r[0])
    return r;
  return fmt == kFmtFp8 ? launch_rowdot_b<Fp8W, 1, EPI>(p, stream)
                        : launch_rowdot_b<Q4W, 1, EPI>(p, stream);
}

} // namespace

const char *rowdot_quant(int epi, RowDotParams &p, int fmt, cudaStream_t stream) {
  switch (epi) {
  case EPI_STORE: return either_format<EPI_STORE>(p, fmt, stream);
  case EPI_ADD: return either_format<EPI_ADD>(p, fmt, stream);
  case EPI_BIAS: return either_format<EPI_BIAS>(p, fmt, stream);
  case EPI_SWIGLU: return either_format<EPI_SWIGLU>(p, fmt, stream);
  case EPI_QKV: return either_format<EPI_QKV>(p, fmt, stream);
  default: return "the quantised projections do not have this epilogue";
  }
}

int rowdot_quant_status() { return take_rowdot_status(); }

} // namespace vxb
