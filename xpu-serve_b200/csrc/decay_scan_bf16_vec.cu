// decay_scan.cuh's kernels for bfloat16 inputs, four entries at a time.
#include "decay_scan.cuh"

namespace xs_decay {

int scan_bf16_vec(const DecayScanArgs& a, int items, cudaStream_t stream) { return launch_scan<__nv_bfloat16, true>(a, items, stream); }

}  // namespace xs_decay
