// Both operands MN-major (weight gradients): instantiations of the tensor-core GEMM for this layout.
#include "gemm_tc.cuh"

namespace dptb {
int gemm_launch_tt(DPTB_GEMM_LAYOUT_ARGS) { DPTB_GEMM_LAYOUT_BODY(true, true) }
}  // namespace dptb
