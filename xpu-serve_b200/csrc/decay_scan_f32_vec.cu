// decay_scan.cuh's kernels for float32 inputs, four entries at a time.
#include "decay_scan.cuh"

namespace xs_decay {

int scan_f32_vec(const DecayScanArgs& a, int items, cudaStream_t stream) { return launch_scan<float, true>(a, items, stream); }

}  // namespace xs_decay
