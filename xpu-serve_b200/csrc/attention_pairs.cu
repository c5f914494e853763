// attention_mma.cu's kernels for value heads of another size than the key heads: keys of 16 to 128 channels with values of
// 32, 64 or 128.
#include "attention_mma.cuh"

namespace xs_attn {

#define XS_PAIRS(GO) \
    GO(16, 32) GO(16, 64) GO(16, 128) GO(32, 64) GO(32, 128) GO(48, 32) GO(48, 64) GO(48, 128) GO(64, 32) GO(64, 128) GO(96, 32) \
    GO(96, 64) GO(96, 128) GO(128, 32) GO(128, 64)

bool pair_supported(int D, int DV) {
#define GO(a, b) if (D == a && DV == b) return true;
    XS_PAIRS(GO)
#undef GO
    return false;
}

int launch_pair(const AttnParams& p, int D, int DV, int max_tiles, int n_seqs, cudaStream_t stream) {
#define GO(a, b) if (D == a && DV == b) return launch<a, b>(p, max_tiles, n_seqs, stream);
    XS_PAIRS(GO)
#undef GO
    return -1;
}

int pair_decode_slots(int D, int DV, int64_t tiles) {
#define GO(a, b) if (D == a && DV == b) return decode_slots<a, b>(tiles);
    XS_PAIRS(GO)
#undef GO
    return 0;
}

}  // namespace xs_attn
