// A K-major, B MN-major (plain matmul, data gradients): instantiations of the tensor-core GEMM for this layout.
#include "gemm_tc.cuh"

namespace dptb {
int gemm_launch_nn(DPTB_GEMM_LAYOUT_ARGS) { DPTB_GEMM_LAYOUT_BODY(false, true) }
}  // namespace dptb
