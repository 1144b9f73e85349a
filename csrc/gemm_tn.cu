// A MN-major, B K-major: instantiations of the tensor-core GEMM for this layout.
#include "gemm_tc.cuh"

namespace dptb {
int gemm_launch_tn(DPTB_GEMM_LAYOUT_ARGS) { DPTB_GEMM_LAYOUT_BODY(true, false) }
}  // namespace dptb
