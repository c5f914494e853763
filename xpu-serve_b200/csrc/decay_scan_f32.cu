// decay_scan.cuh's kernels for float32 inputs, one entry at a time.
#include "decay_scan.cuh"

namespace xs_decay {

int scan_f32(const DecayScanArgs& a, int items, cudaStream_t stream) { return launch_scan<float, false>(a, items, stream); }

}  // namespace xs_decay
