// Linear-attention memories whose rows (key channels) decay each at a rate of their own, token by token: per (sequence, head)
// S [D, E], float32, zero at a sequence's start, with a_t [D] in (0, 1] given in float32:
//
//   read behind the write:   S_t = diag(a_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T (q_t * q_scale)
//   bonus (read before it):  o_t = (S_(t-1) + diag(u) k_t v_t^T)^T (q_t * q_scale),   then S_t as above
//
// q, k and v come in the activation type; everything else is float32. A CTA walks one (sequence, head, block of 32 CPL value
// columns) in order: WARPS warps, warp g holding NR neighbouring rows of the block's columns in registers (a lane CPL columns),
// so that a token's k, a and q come from shared memory four rows at a time, as broadcasts that serve CPL columns each. Tokens
// are staged kBatch at a time: the next ones are fetched into registers before the current ones are walked and go to the other of
// two shared buffers behind them. The warps' partial sums of a token's output are added in the order of the warps.
//
// Where one CTA holds all columns of a head, the head's output is finished there: divided by its root mean square, times a
// weight, times silu of a gate's logits, in the activation type. Otherwise the float32 sums go to y.
//
// Long pieces of a prompt run as chunks side by side in three launches: every chunk from the empty state (leaving its end
// state and the product of its decays), a carry over each sequence's chunks in order (S <- product S + local, which is what the
// recurrence unrolls to; each chunk is left with the state it starts from), and the chunks again from their true states.
#pragma once

#include <math.h>

#include "common.cuh"

namespace xs_decay {

constexpr int kBatch = 8;        // tokens staged at a time

enum ScanMode : int { kSequences = 0, kChunkLocal = 1, kChunkFinal = 2 };

struct DecayScanArgs {
    const void* q;               // head h's D values at q + row * ld_q + h * D; k and v likewise (v: h * E)
    const void* k;
    const void* v;
    int64_t ld_q, ld_k, ld_v;
    const float* decay;          // [T, H * D]
    const float* bonus;          // [H, D] or null
    float* state;                // [slots, H, D, E]
    const int32_t* cu_seqlens;   // [sequences + 1]
    const int32_t* slots;        // [sequences]
    float* y;                    // [T, H * E], or null: finished into out
    void* out;                   // [T, H * E] in the activation type, rows `ld_out` apart
    int64_t ld_out;
    const float* norm_w;         // [H * E]
    const void* gate;            // logits, head h's E values at gate + row * ld_gate + h * E
    int64_t ld_gate;
    const int32_t* chunks;       // [n, 3] (sequence, first token, tokens), or null
    float* chunk_state;          // [n, H, D, E]
    float* chunk_decay;          // [n, H, D]
    int H, D, E, mode, vec;      // vec: q, k, v and decay rows may be read four entries at a time
    float q_scale, eps;
};

// Four neighbouring entries as they come from memory (16-byte aligned float32, 8-byte aligned bfloat16), zeros where not `there`.
__device__ __forceinline__ uint4 load_quad(const float* p, bool there) {
    return there ? *reinterpret_cast<const uint4*>(p) : make_uint4(0u, 0u, 0u, 0u);
}
__device__ __forceinline__ uint4 load_quad(const __nv_bfloat16* p, bool there) {
    const uint2 r = there ? *reinterpret_cast<const uint2*>(p) : make_uint2(0u, 0u);
    return make_uint4(r.x, r.y, 0u, 0u);
}
template <typename T>
__device__ __forceinline__ float4 quad_floats(const uint4& r) {
    if constexpr (sizeof(T) == 4) {
        return make_float4(__uint_as_float(r.x), __uint_as_float(r.y), __uint_as_float(r.z), __uint_as_float(r.w));
    } else {                     // a bfloat16 is the upper half of the float with its value
        return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xffff0000u), __uint_as_float(r.y << 16),
                           __uint_as_float(r.y & 0xffff0000u));
    }
}

// a lane's CPL neighbouring columns
template <int CPL>
__device__ __forceinline__ void load_cols(const float* p, float (&v)[CPL], int valid, bool vec) {
    if (vec && valid >= CPL) {
        if constexpr (CPL == 4) {
            const float4 r = *reinterpret_cast<const float4*>(p);
            v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
        } else if constexpr (CPL == 2) {
            const float2 r = *reinterpret_cast<const float2*>(p);
            v[0] = r.x; v[1] = r.y;
        } else {
            v[0] = p[0];
        }
    } else {
#pragma unroll
        for (int j = 0; j < CPL; ++j) v[j] = j < valid ? p[j] : 0.0f;
    }
}
template <int CPL>
__device__ __forceinline__ void store_cols(float* p, const float (&v)[CPL], int valid, bool vec) {
    if (vec && valid >= CPL) {
        if constexpr (CPL == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        else if constexpr (CPL == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
        else p[0] = v[0];
    } else {
#pragma unroll
        for (int j = 0; j < CPL; ++j)
            if (j < valid) p[j] = v[j];
    }
}

// In front of a rounding to bfloat16 the fast exponential and division do; float32 outputs take the exact ones.
template <typename T>
__device__ __forceinline__ float silu_gate(float z) {
    if constexpr (sizeof(T) == 4) return z / (1.0f + expf(-z));
    else return __fdividef(z, 1.0f + __expf(-z));
}

// What a launch computes: the states alone (a chunk's first pass), or outputs, read behind the write or before it with a bonus.
enum ScanKind : int { kStates = 0, kReadBehind = 1, kReadBonus = 2 };

// CTAs an SM that the registers are bounded for.
constexpr int scan_ctas(int NR, int WARPS, int CPL) { return WARPS == 8 ? (NR * CPL <= 16 ? 3 : 2) : NR * CPL <= 16 ? 6 : NR * CPL <= 32 ? 5 : 4; }

// VEC: rows of q, k, v and decay are read four entries at a time (their sizes and places allow it); otherwise one at a time.
template <typename T, int NR, int WARPS, int CPL, int KIND, bool VEC>
__global__ void __launch_bounds__(WARPS * 32, scan_ctas(NR, WARPS, CPL)) decay_scan_kernel(const DecayScanArgs a) {
    constexpr bool outputs = KIND != kStates, BONUS = KIND == kReadBonus;
    extern __shared__ __align__(16) float smem[];
    constexpr int DP = NR * WARPS, COLS = 32 * CPL, ROW = 3 * DP + COLS, THREADS = WARPS * 32;
    constexpr int STEP = VEC ? 4 : 1;                 // entries of a staged row that a thread moves together
    constexpr int PIECES = ROW / STEP, NL = (kBatch * PIECES + THREADS - 1) / THREADS, TPW = kBatch / WARPS;
    static_assert(kBatch % WARPS == 0, "a warp finishes whole tokens");
    const int D = a.D, E = a.E;
    float* stage = smem;                              // [2][kBatch][ROW]: q, k, a (zeros from D on), v
    float* part = smem + 2 * kBatch * ROW;            // [2][kBatch][WARPS][COLS]
    float* bonus = part + 2 * kBatch * WARPS * COLS;  // [DP]
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, g = threadIdx.x >> 5;
    const int h = blockIdx.y, c0 = blockIdx.x * COLS, col = c0 + lane * CPL;
    const int valid = E - col;                        // of this lane's columns, those that exist
    const bool cvec = E % CPL == 0;
    int t0, n, slot;
    if (a.mode == kSequences) {
        t0 = a.cu_seqlens[blockIdx.z];
        n = a.cu_seqlens[blockIdx.z + 1] - t0;
        slot = a.slots[blockIdx.z];
    } else {
        const int32_t* ch = a.chunks + 3 * (int64_t)blockIdx.z;
        t0 = ch[1];
        n = ch[2];
        slot = 0;
    }
    if (n <= 0) return;
    const T *qp = (const T*)a.q + h * D, *kp = (const T*)a.k + h * D, *vp = (const T*)a.v + h * E + c0;
    const float* ap = a.decay + h * D;

    // this thread's pieces of the staged tokens: entries j .. j + STEP - 1 of token tt's row
    uint4 quads[VEC ? NL : 1];
    float ones[VEC ? 1 : NL];
    auto fetch = [&](int b0) {
#pragma unroll
        for (int u = 0; u < NL; ++u) {
            const int e = threadIdx.x + u * THREADS;
            const int tt = e / PIECES, j = (e - tt * PIECES) * STEP;
            const bool token_there = tt < kBatch && b0 + tt < n;
            const int64_t t = t0 + b0 + tt;
            if constexpr (VEC) {
                if (j < DP) quads[u] = load_quad(qp + t * a.ld_q + j, token_there && outputs && j < D);
                else if (j < 2 * DP) quads[u] = load_quad(kp + t * a.ld_k + (j - DP), token_there && j - DP < D);
                else if (j < 3 * DP) quads[u] = load_quad(ap + t * ((int64_t)a.H * D) + (j - 2 * DP), token_there && j - 2 * DP < D);
                else quads[u] = load_quad(vp + t * a.ld_v + (j - 3 * DP), token_there && c0 + (j - 3 * DP) < E);
            } else {
                float v = 0.0f;
                if (token_there) {
                    if (j < DP) {
                        if (outputs && j < D) v = to_f32(qp[t * a.ld_q + j]);
                    } else if (j < 2 * DP) {
                        if (j - DP < D) v = to_f32(kp[t * a.ld_k + (j - DP)]);
                    } else if (j < 3 * DP) {
                        if (j - 2 * DP < D) v = ap[t * ((int64_t)a.H * D) + (j - 2 * DP)];
                    } else if (c0 + (j - 3 * DP) < E) {
                        v = to_f32(vp[t * a.ld_v + (j - 3 * DP)]);
                    }
                }
                ones[u] = v;
            }
        }
    };
    auto put = [&](float* buf) {
#pragma unroll
        for (int u = 0; u < NL; ++u) {
            const int e = threadIdx.x + u * THREADS;
            if (kBatch * PIECES % THREADS != 0 && e >= kBatch * PIECES) continue;
            const int tt = e / PIECES, j = (e - tt * PIECES) * STEP;
            if constexpr (VEC) {
                float4 v = (j >= 2 * DP && j < 3 * DP) ? quad_floats<float>(quads[u]) : quad_floats<T>(quads[u]);
                if (j < DP) v.x *= a.q_scale, v.y *= a.q_scale, v.z *= a.q_scale, v.w *= a.q_scale;
                *reinterpret_cast<float4*>(buf + tt * ROW + j) = v;
            } else {
                buf[tt * ROW + j] = j < DP ? ones[u] * a.q_scale : ones[u];
            }
        }
    };

    if constexpr (BONUS)
        for (int i = threadIdx.x; i < DP; i += THREADS) bonus[i] = i < D ? a.bonus[h * D + i] : 0.0f;
    pdl_wait();
    float S[NR][CPL];
    {
        const float* from = a.mode == kSequences ? a.state + (((int64_t)slot * a.H + h) * D) * E
                            : a.mode == kChunkFinal ? a.chunk_state + (((int64_t)blockIdx.z * a.H + h) * D) * E : nullptr;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int r = g * NR + i;
            load_cols<CPL>(from + (int64_t)r * E + col, S[i], from != nullptr && r < D ? valid : 0, cvec);
        }
    }
    fetch(0);
    put(stage);
    __syncthreads();

    float product = 1.0f;        // (a chunk's first pass) of the decays of row g NR + lane
    auto token = [&](const float* q, float* pp_t) {
        const float4* q4 = reinterpret_cast<const float4*>(q + g * NR);
        const float4* k4 = reinterpret_cast<const float4*>(q + DP + g * NR);
        const float4* a4 = reinterpret_cast<const float4*>(q + 2 * DP + g * NR);
        float v[CPL], acc0[CPL], acc1[CPL];
        load_cols<CPL>(q + 3 * DP + lane * CPL, v, CPL, true);
#pragma unroll
        for (int j = 0; j < CPL; ++j) acc0[j] = acc1[j] = 0.0f;
#pragma unroll
        for (int i = 0; i < NR / 4; ++i) {
            const float4 kk4 = k4[i], aa4 = a4[i];
            const float kk[4] = {kk4.x, kk4.y, kk4.z, kk4.w}, aa[4] = {aa4.x, aa4.y, aa4.z, aa4.w};
            float qq[4] = {0.0f, 0.0f, 0.0f, 0.0f}, uu[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            if constexpr (BONUS) {
                const float4 uu4 = *reinterpret_cast<const float4*>(bonus + g * NR + 4 * i);
                uu[0] = uu4.x; uu[1] = uu4.y; uu[2] = uu4.z; uu[3] = uu4.w;
            }
            if (outputs) {
                const float4 qq4 = q4[i];
                qq[0] = qq4.x; qq[1] = qq4.y; qq[2] = qq4.z; qq[3] = qq4.w;
            }
#pragma unroll
            for (int m = 0; m < 4; ++m) {
#pragma unroll
                for (int j = 0; j < CPL; ++j) {
                    float& s = S[4 * i + m][j];
                    float& acc = m & 1 ? acc1[j] : acc0[j];
                    const float kv = kk[m] * v[j];
                    if (BONUS && outputs) acc = fmaf(fmaf(uu[m], kv, s), qq[m], acc);
                    s = fmaf(aa[m], s, kv);
                    if (!BONUS && outputs) acc = fmaf(s, qq[m], acc);
                }
            }
        }
        if (outputs) {
            float o[CPL];
#pragma unroll
            for (int j = 0; j < CPL; ++j) o[j] = acc0[j] + acc1[j];
            store_cols<CPL>(pp_t + g * COLS + lane * CPL, o, CPL, true);
        } else if (lane < NR) {
            product *= q[2 * DP + g * NR + lane];
        }
    };

    float wn[CPL];
    const bool finish = outputs && a.y == nullptr;
    if (finish) load_cols<CPL>(a.norm_w + (int64_t)h * E + col, wn, valid, false);
    int which = 0;
    for (int b0 = 0; b0 < n; b0 += kBatch) {
        const int cnt = min(kBatch, n - b0);
        const bool more = b0 + kBatch < n;
        if (more) fetch(b0 + kBatch);
        // the gates of the tokens that this warp finishes, asked for before the walk
        T gates[TPW][CPL];
        if (finish) {
#pragma unroll
            for (int u = 0; u < TPW; ++u) {
                const int tt = g + u * WARPS;
                const T* gp = (const T*)a.gate + (int64_t)(t0 + b0 + tt) * a.ld_gate + (int64_t)h * E + col;
#pragma unroll
                for (int j = 0; j < CPL; ++j) gates[u][j] = tt < cnt && j < valid ? gp[j] : from_f32<T>(0.0f);
            }
        }
        const float* buf = stage + which * kBatch * ROW;
        float* pp = part + which * kBatch * WARPS * COLS;
        if (cnt == kBatch) {
#pragma unroll(NR * CPL <= 32 && !BONUS ? 2 : 1)
            for (int tt = 0; tt < kBatch; ++tt) token(buf + tt * ROW, pp + tt * WARPS * COLS);
        } else {
            for (int tt = 0; tt < cnt; ++tt) token(buf + tt * ROW, pp + tt * WARPS * COLS);
        }
        if (more) put(stage + (which ^ 1) * kBatch * ROW);
        __syncthreads();
        if (outputs) {
#pragma unroll
            for (int u = 0; u < TPW; ++u) {
                const int tt = g + u * WARPS;
                if (tt >= cnt) break;
                float o[CPL];
#pragma unroll
                for (int j = 0; j < CPL; ++j) o[j] = 0.0f;
#pragma unroll
                for (int w = 0; w < WARPS; ++w) {
                    float p[CPL];
                    load_cols<CPL>(pp + (tt * WARPS + w) * COLS + lane * CPL, p, CPL, true);
#pragma unroll
                    for (int j = 0; j < CPL; ++j) o[j] += p[j];
                }
                const int64_t t = t0 + b0 + tt;
                if (!finish) {
                    store_cols<CPL>(a.y + (t * a.H + h) * E + col, o, valid, cvec);
                    continue;
                }
                float ss = 0.0f;
#pragma unroll
                for (int j = 0; j < CPL; ++j) ss = fmaf(o[j], o[j], ss);
                const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)E + a.eps);
                T* op = (T*)a.out + t * a.ld_out + (int64_t)h * E + col;
                float f[CPL];
#pragma unroll
                for (int j = 0; j < CPL; ++j) f[j] = o[j] * inv * wn[j] * silu_gate<T>(to_f32(gates[u][j]));
                if constexpr (CPL >= 2 && sizeof(T) == 2) {
                    if (cvec && a.ld_out % 2 == 0 && valid >= CPL) {
#pragma unroll
                        for (int j = 0; j < CPL; j += 2) *reinterpret_cast<__nv_bfloat162*>(op + j) = __floats2bfloat162_rn(f[j], f[j + 1]);
                        continue;
                    }
                }
#pragma unroll
                for (int j = 0; j < CPL; ++j)
                    if (j < valid) op[j] = from_f32<T>(f[j]);
            }
        }
        which ^= 1;
    }
    if (a.mode != kChunkFinal) {
        float* to = a.mode == kSequences ? a.state + (((int64_t)slot * a.H + h) * D) * E
                                         : a.chunk_state + (((int64_t)blockIdx.z * a.H + h) * D) * E;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int r = g * NR + i;
            store_cols<CPL>(to + (int64_t)r * E + col, S[i], r < D ? valid : 0, cvec);
        }
        if (a.mode == kChunkLocal && blockIdx.x == 0 && lane < NR && g * NR + lane < D)
            a.chunk_decay[((int64_t)blockIdx.z * a.H + h) * D + g * NR + lane] = product;
    }
}

template <typename T, int NR, int WARPS, int CPL, bool VEC>
void launch_as(const DecayScanArgs& a, int items, cudaStream_t stream) {
    constexpr int ROW = 3 * NR * WARPS + 32 * CPL;
    const size_t smem = (size_t)(2 * kBatch * ROW + 2 * kBatch * WARPS * 32 * CPL + NR * WARPS) * sizeof(float);
    const dim3 grid(ceil_div_i(a.E, 32 * CPL), a.H, items);
    const auto kernel = a.mode == kChunkLocal ? decay_scan_kernel<T, NR, WARPS, CPL, kStates, VEC>
                        : a.bonus != nullptr  ? decay_scan_kernel<T, NR, WARPS, CPL, kReadBonus, VEC>
                                              : decay_scan_kernel<T, NR, WARPS, CPL, kReadBehind, VEC>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    xs_launch(kernel, grid, dim3(WARPS * 32), smem, stream, a);
}

// columns a lane: as few as hold a head's columns in one CTA, at most what the rows leave registers for
inline int columns_per_lane(int D, int E) { return E <= 32 ? 1 : E <= 64 || D > 128 ? 2 : 4; }

template <typename T, bool VEC>
int launch_scan(const DecayScanArgs& a, int items, cudaStream_t stream) {
    const int cpl = columns_per_lane(a.D, a.E);
#define XS_GO(NR, WARPS)                                           \
    do {                                                           \
        if (cpl == 1) launch_as<T, NR, WARPS, 1, VEC>(a, items, stream); \
        else if (cpl == 2) launch_as<T, NR, WARPS, 2, VEC>(a, items, stream); \
        else launch_as<T, NR, WARPS, 4, VEC>(a, items, stream);    \
    } while (0)
    if (a.D <= 32) XS_GO(8, 4);
    else if (a.D <= 64) XS_GO(16, 4);
    else if (a.D <= 128) XS_GO(16, 8);
    else if (cpl == 1) launch_as<T, 32, 8, 1, VEC>(a, items, stream);
    else launch_as<T, 32, 8, 2, VEC>(a, items, stream);
#undef XS_GO
    return 0;
}

// The four groups of instances are compiled side by side (decay_scan_*.cu).
int scan_f32(const DecayScanArgs& a, int items, cudaStream_t stream);          // one entry at a time
int scan_f32_vec(const DecayScanArgs& a, int items, cudaStream_t stream);
int scan_bf16(const DecayScanArgs& a, int items, cudaStream_t stream);
int scan_bf16_vec(const DecayScanArgs& a, int items, cudaStream_t stream);

}  // namespace xs_decay
