// x W^T: both operands K-major (every forward product): instantiations of the tensor-core GEMM for this layout.
#include "gemm_tc.cuh"

namespace dptb {
int gemm_launch_nt(DPTB_GEMM_LAYOUT_ARGS) { DPTB_GEMM_LAYOUT_BODY(false, false) }
}  // namespace dptb

using namespace dptb;

// Role timers (see DPTB_GEMM_PROFILE): copies [256][12] counters out and zeroes them; -5 when not compiled in.
extern "C" int dptb_gemm_profile_read(unsigned long long* out) {
#ifdef DPTB_GEMM_PROFILE
  int rc = (int)cudaMemcpyFromSymbol(out, g_gemm_prof, sizeof(unsigned long long) * 256 * kProfSlots);
  if (rc) return rc;
  static unsigned long long zeros[256 * kProfSlots];
  return (int)cudaMemcpyToSymbol(g_gemm_prof, zeros, sizeof(zeros));
#else
  (void)out;
  return kErrUnsupported;
#endif
}
