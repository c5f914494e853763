// decay_scan.cuh's kernels for bfloat16 inputs, one entry at a time.
#include "decay_scan.cuh"

namespace xs_decay {

int scan_bf16(const DecayScanArgs& a, int items, cudaStream_t stream) { return launch_scan<__nv_bfloat16, false>(a, items, stream); }

}  // namespace xs_decay
