// All-gather form of the tensor-core GEMM (A read in place from every rank's shard).
#include "gemm_tc.cuh"

namespace dptb {
int gemm_launch_ag(int bn, const TmapSet& peers, const CUtensorMap& tmB, const GemmParams& p, cudaStream_t stream) {
  return bn == 256 ? launch_tc_ag<256, 4>(peers, tmB, p, stream) : launch_tc_ag<128, 6>(peers, tmB, p, stream);
}
}  // namespace dptb
