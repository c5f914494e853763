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
#include <math.h>

#include "common.cuh"

namespace {

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

// Four neighbouring entries as they come from memory: n of them exist, the others are zero.
__device__ __forceinline__ uint4 load_quad(const float* p, int n, bool vec) {
    if (vec) return n > 0 ? *reinterpret_cast<const uint4*>(p) : make_uint4(0u, 0u, 0u, 0u);
    return make_uint4(n > 0 ? __float_as_uint(p[0]) : 0u, n > 1 ? __float_as_uint(p[1]) : 0u, n > 2 ? __float_as_uint(p[2]) : 0u,
                      n > 3 ? __float_as_uint(p[3]) : 0u);
}
__device__ __forceinline__ uint4 load_quad(const __nv_bfloat16* p, int n, bool vec) {
    if (vec) {
        const uint2 r = n > 0 ? *reinterpret_cast<const uint2*>(p) : make_uint2(0u, 0u);
        return make_uint4(r.x, r.y, 0u, 0u);
    }
    const unsigned short* u = reinterpret_cast<const unsigned short*>(p);
    const unsigned e0 = n > 0 ? u[0] : 0u, e1 = n > 1 ? u[1] : 0u, e2 = n > 2 ? u[2] : 0u, e3 = n > 3 ? u[3] : 0u;
    return make_uint4(e0 | e1 << 16, e2 | e3 << 16, 0u, 0u);
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

template <typename T, int NR, int WARPS, int CPL, int KIND>
__global__ void __launch_bounds__(WARPS * 32, scan_ctas(NR, WARPS, CPL)) decay_scan_kernel(const DecayScanArgs a) {
    constexpr bool outputs = KIND != kStates, BONUS = KIND == kReadBonus;
    extern __shared__ __align__(16) float smem[];
    constexpr int DP = NR * WARPS, COLS = 32 * CPL, ROW = 3 * DP + COLS, THREADS = WARPS * 32;
    constexpr int G4 = ROW / 4, NL = (kBatch * G4 + THREADS - 1) / THREADS, TPW = kBatch / WARPS;
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
    const bool vec = a.vec != 0;
    const T *qp = (const T*)a.q + h * D, *kp = (const T*)a.k + h * D, *vp = (const T*)a.v + h * E + c0;
    const float* ap = a.decay + h * D;

    // the staged quads of this thread: which part of a token's row, which token of a batch
    uint4 fetched[NL];
    auto fetch = [&](int b0) {
#pragma unroll
        for (int u = 0; u < NL; ++u) {
            const int e = threadIdx.x + u * THREADS;
            const int tt = e / G4, j = (e - tt * G4) * 4;
            const int64_t t = t0 + b0 + tt;
            const bool there = tt < kBatch && b0 + tt < n;
            if (j < DP) fetched[u] = load_quad(qp + t * a.ld_q + j, there && outputs ? D - j : 0, vec);
            else if (j < 2 * DP) fetched[u] = load_quad(kp + t * a.ld_k + (j - DP), there ? D - (j - DP) : 0, vec);
            else if (j < 3 * DP) fetched[u] = load_quad(ap + t * ((int64_t)a.H * D) + (j - 2 * DP), there ? D - (j - 2 * DP) : 0, vec);
            else fetched[u] = load_quad(vp + t * a.ld_v + (j - 3 * DP), there ? E - c0 - (j - 3 * DP) : 0, vec);
        }
    };
    auto put = [&](float* buf) {
#pragma unroll
        for (int u = 0; u < NL; ++u) {
            const int e = threadIdx.x + u * THREADS;
            if (kBatch * G4 % THREADS == 0 || e < kBatch * G4) {
                const int tt = e / G4, j = (e - tt * G4) * 4;
                float4 v = (j >= 2 * DP && j < 3 * DP) ? quad_floats<float>(fetched[u]) : quad_floats<T>(fetched[u]);
                if (j < DP) v.x *= a.q_scale, v.y *= a.q_scale, v.z *= a.q_scale, v.w *= a.q_scale;
                *reinterpret_cast<float4*>(buf + tt * ROW + j) = v;
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

template <typename T, int NR, int WARPS, int CPL>
void launch_as(const DecayScanArgs& a, int items, cudaStream_t stream) {
    constexpr int ROW = 3 * NR * WARPS + 32 * CPL;
    const size_t smem = (size_t)(2 * kBatch * ROW + 2 * kBatch * WARPS * 32 * CPL + NR * WARPS) * sizeof(float);
    const dim3 grid(ceil_div_i(a.E, 32 * CPL), a.H, items);
    const auto kernel = a.mode == kChunkLocal ? decay_scan_kernel<T, NR, WARPS, CPL, kStates>
                        : a.bonus != nullptr  ? decay_scan_kernel<T, NR, WARPS, CPL, kReadBonus>
                                              : decay_scan_kernel<T, NR, WARPS, CPL, kReadBehind>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    xs_launch(kernel, grid, dim3(WARPS * 32), smem, stream, a);
}

// columns a lane: as few as hold a head's columns in one CTA, at most what the rows leave registers for
int columns_per_lane(int D, int E) { return E <= 32 ? 1 : E <= 64 || D > 128 ? 2 : 4; }

template <typename T>
int launch_scan(const DecayScanArgs& a, int items, cudaStream_t stream) {
    const int cpl = columns_per_lane(a.D, a.E);
#define XS_GO(NR, WARPS)                                           \
    do {                                                           \
        if (cpl == 1) launch_as<T, NR, WARPS, 1>(a, items, stream); \
        else if (cpl == 2) launch_as<T, NR, WARPS, 2>(a, items, stream); \
        else launch_as<T, NR, WARPS, 4>(a, items, stream);         \
    } while (0)
    if (a.D <= 32) XS_GO(8, 4);
    else if (a.D <= 64) XS_GO(16, 4);
    else if (a.D <= 128) XS_GO(16, 8);
    else if (cpl == 1) launch_as<T, 32, 8, 1>(a, items, stream);
    else launch_as<T, 32, 8, 2>(a, items, stream);
#undef XS_GO
    return 0;
}

}  // namespace

// 1 when xs_decay_scan finishes a head's output itself (norm, weight, gate).
XS_API int xs_decay_scan_finishes(int D, int E) { return E <= 32 * columns_per_lane(D, E) ? 1 : 0; }

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
    DecayScanArgs a{q, k, v, ld_q, ld_k, ld_v, decay, bonus, state, cu_seqlens, slots, y, out, ld_out, norm_w, gate, ld_gate,
                    chunks, chunk_state, chunk_decay, H, D, E, kSequences, 0, q_scale, eps};
    a.vec = D % 4 == 0 && E % 4 == 0 && ld_q % 4 == 0 && ld_k % 4 == 0 && ld_v % 4 == 0 &&
            ((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)decay) % 16 == 0;
    if (chunks == nullptr) {
        XS_DISPATCH_DTYPE(dtype, TT, launch_scan<TT>(a, n_seqs, stream));
        XS_LAUNCH_CHECK("decay_scan");
        return 0;
    }
    a.mode = kChunkLocal;
    XS_DISPATCH_DTYPE(dtype, TT, launch_scan<TT>(a, n_chunks, stream));
    XS_LAUNCH_CHECK("decay_scan (chunks, local)");
    xs_launch(decay_carry_kernel, dim3(ceil_div_i((int64_t)D * E, 256), H, n_seqs), dim3(256), 0, stream, state, slots, first_chunk,
              chunk_state, (const float*)chunk_decay, H, D, E);
    XS_LAUNCH_CHECK("decay_carry");
    a.mode = kChunkFinal;
    XS_DISPATCH_DTYPE(dtype, TT, launch_scan<TT>(a, n_chunks, stream));
    XS_LAUNCH_CHECK("decay_scan (chunks, final)");
    return 0;
}
