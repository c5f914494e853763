// The interface of decay_scan.cuh's kernels, and the carry between chunks.
#include "decay_scan.cuh"

using namespace xs_decay;

namespace {

// Per sequence, in the order of its chunks: the chunk's local end state gives way to the state the chunk starts from, and the
// running state moves on by the chunk's product of decays times itself plus the local end state; the last one is the
// sequence's new state. Eight chunks' loads are in flight together.
__global__ void decay_carry_kernel(float* __restrict__ state, const int32_t* __restrict__ slots, const int32_t* __restrict__ first_chunk,
                                   float* __restrict__ chunk_state, const float* __restrict__ chunk_decay, int H, int D, int E) {
    pdl_launch_dependents();
    const int seq = blockIdx.z, h = blockIdx.y;
    const int c_lo = first_chunk[seq], c_hi = first_chunk[seq + 1];
    const int64_t per_head = (int64_t)D * E;
    const int64_t e = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_wait();
    if (c_lo >= c_hi || e >= per_head) return;
    const int d = (int)(e / E);
    float* st = state + ((int64_t)slots[seq] * H + h) * per_head + e;
    float run = *st;
    for (int c = c_lo; c < c_hi; c += 8) {
        float local[8], f[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int64_t at = (int64_t)min(c + j, c_hi - 1) * H + h;
            local[j] = chunk_state[at * per_head + e];
            f[j] = chunk_decay[at * D + d];
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (c + j < c_hi) {
                chunk_state[((int64_t)(c + j) * H + h) * per_head + e] = run;
                run = fmaf(f[j], run, local[j]);
            }
        }
    }
    *st = run;
}

int scan(const DecayScanArgs& a, int items, int dtype, cudaStream_t stream) {
    if (dtype == XS_F32) return a.vec ? scan_f32_vec(a, items, stream) : scan_f32(a, items, stream);
    return a.vec ? scan_bf16_vec(a, items, stream) : scan_bf16(a, items, stream);
}

}  // namespace

// 1 when xs_decay_scan finishes a head's output itself (norm, weight, gate).
XS_API int xs_decay_scan_finishes(int D, int E) { return E <= 32 * columns_per_lane(D, E) ? 1 : 0; }

// CTAs that run at one time on an SM, by the registers they are bounded for.
XS_API int xs_decay_scan_ctas(int D, int E) {
    const int cpl = columns_per_lane(D, E);
    return D <= 32 ? scan_ctas(8, 4, cpl) : D <= 64 ? scan_ctas(16, 4, cpl) : D <= 128 ? scan_ctas(16, 8, cpl) : scan_ctas(32, 8, cpl);
}

// CTAs of one (sequence or chunk).
XS_API int xs_decay_scan_blocks(int H, int D, int E) { return H * ceil_div_i(E, 32 * columns_per_lane(D, E)); }

// q, k, v: rows `ld_*` apart in the element type `dtype`; decay [T, H * D], state [slots, H, D, E] float32. y [T, H * E] float32,
// or null with out / norm_w / gate: the finished heads. With `chunks` ([n_chunks, 3] int32: sequence, first token, tokens;
// `first_chunk` [n_seqs + 1]; `chunk_state` [n_chunks, H, D, E], `chunk_decay` [n_chunks, H, D] float32) the chunks run side by
// side in three launches.
XS_API int xs_decay_scan(const void* q, int64_t ld_q, const void* k, int64_t ld_k, const void* v, int64_t ld_v, const float* decay,
                         const float* bonus, float* state, const int32_t* cu_seqlens, const int32_t* slots, float* y, void* out,
                         int64_t ld_out, const float* norm_w, const void* gate, int64_t ld_gate, int n_seqs, int H, int D, int E,
                         float q_scale, float eps, int dtype, const int32_t* chunks, const int32_t* first_chunk, int n_chunks,
                         float* chunk_state, float* chunk_decay, cudaStream_t stream) {
    if (n_seqs == 0) return 0;
    XS_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && H > 0 && H <= 65535 && D > 0 && D <= 256 && E > 0,
               "decay_scan: %d sequences, %d heads of %d x %d (keys of at most 256)", n_seqs, H, D, E);
    XS_REQUIRE(ld_q >= (int64_t)H * D && ld_k >= (int64_t)H * D && ld_v >= (int64_t)H * E, "decay_scan: rows shorter than %d heads", H);
    XS_REQUIRE(y != nullptr || (xs_decay_scan_finishes(D, E) && out != nullptr && norm_w != nullptr && gate != nullptr &&
                                ld_out >= (int64_t)H * E && ld_gate >= (int64_t)H * E),
               "decay_scan: heads of %d values cannot be finished here", E);
    XS_REQUIRE(chunks == nullptr || (first_chunk != nullptr && chunk_state != nullptr && chunk_decay != nullptr && n_chunks > 0 && n_chunks <= 65535),
               "decay_scan: %d chunks without their scratch", n_chunks);
    XS_REQUIRE(dtype == XS_F32 || dtype == XS_BF16, "decay_scan: unknown element type code %d", dtype);
    DecayScanArgs a{q, k, v, ld_q, ld_k, ld_v, decay, bonus, state, cu_seqlens, slots, y, out, ld_out, norm_w, gate, ld_gate,
                    chunks, chunk_state, chunk_decay, H, D, E, kSequences, 0, q_scale, eps};
    a.vec = D % 4 == 0 && E % 4 == 0 && ld_q % 4 == 0 && ld_k % 4 == 0 && ld_v % 4 == 0 &&
            ((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)decay) % 16 == 0;
    if (chunks == nullptr) {
        scan(a, n_seqs, dtype, stream);
        XS_LAUNCH_CHECK("decay_scan");
        return 0;
    }
    a.mode = kChunkLocal;
    scan(a, n_chunks, dtype, stream);
    XS_LAUNCH_CHECK("decay_scan (chunks, local)");
    xs_launch(decay_carry_kernel, dim3(ceil_div_i((int64_t)D * E, 256), H, n_seqs), dim3(256), 0, stream, state, slots, first_chunk,
              chunk_state, (const float*)chunk_decay, H, D, E);
    XS_LAUNCH_CHECK("decay_carry");
    a.mode = kChunkFinal;
    scan(a, n_chunks, dtype, stream);
    XS_LAUNCH_CHECK("decay_scan (chunks, final)");
    return 0;
}
