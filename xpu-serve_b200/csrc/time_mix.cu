// What feeds the recurrences of decay_scan.cu beside the plain projections:
//
//   token_mix      out[s, t, c] = x[t, c] + (x[t - 1, c] - x[t, c]) * mu[s, c]: several mixes of every token with the one before it
//                  in its sequence (zeros before the first); the previous step's last row comes from the sequence's state
//   low_rank_decay out[t, c] = g(sum_j w[c, j] f(z[t, j]) + bias[c]): decays from a low-rank hidden vector, all float32.
//                  f: nothing or tanh; g: exp(-exp(v)), or sigmoid(v)^power
//
// Float32 sums in an order that depends on the sizes alone, whatever else is in the batch.
#include <math.h>

#include "common.cuh"

namespace {

// A block a token (and a run of columns). Every first token of a sequence reads the sequence's state and, having read it,
// leaves the sequence's last row of this step there: nobody else touches that row.
template <typename T>
__global__ void token_mix_kernel(const T* __restrict__ x, int64_t ldx, T* __restrict__ state, const float* __restrict__ mu, T* __restrict__ out,
                                 const int32_t* __restrict__ seq_of_token, const int32_t* __restrict__ cu_seqlens,
                                 const int32_t* __restrict__ slots, int64_t plane, int W, int mixes) {
    pdl_launch_dependents();
    const int t = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= W) return;
    const int seq = seq_of_token[t];
    const int first = cu_seqlens[seq], last = cu_seqlens[seq + 1] - 1;
    T* st = state + (int64_t)slots[seq] * W + c;
    pdl_wait();
    const float cur = to_f32(x[(int64_t)t * ldx + c]);
    float prev;
    if (t > first) prev = to_f32(x[(int64_t)(t - 1) * ldx + c]);
    else {
        prev = to_f32(*st);
        *st = x[(int64_t)last * ldx + c];
    }
    for (int s = 0; s < mixes; ++s) out[s * plane + (int64_t)t * W + c] = from_f32<T>(fmaf(prev - cur, mu[(int64_t)s * W + c], cur));
}

// bfloat16 rows in 16-byte pieces.
__global__ void token_mix_vec_kernel(const __nv_bfloat16* __restrict__ x, int64_t ldx, __nv_bfloat16* __restrict__ state,
                                     const float* __restrict__ mu, __nv_bfloat16* __restrict__ out, const int32_t* __restrict__ seq_of_token,
                                     const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ slots, int64_t plane, int W,
                                     int mixes) {
    pdl_launch_dependents();
    const int t = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
    if (c >= W) return;
    const int seq = seq_of_token[t];
    const int first = cu_seqlens[seq], last = cu_seqlens[seq + 1] - 1;
    uint4* st = reinterpret_cast<uint4*>(state + (int64_t)slots[seq] * W + c);
    pdl_wait();
    const uint4 cur4 = *reinterpret_cast<const uint4*>(x + (int64_t)t * ldx + c);
    uint4 prev4;
    if (t > first) prev4 = *reinterpret_cast<const uint4*>(x + (int64_t)(t - 1) * ldx + c);
    else {
        prev4 = *st;
        *st = *reinterpret_cast<const uint4*>(x + (int64_t)last * ldx + c);
    }
    float cur[8], step[8];
    {
        const __nv_bfloat162 *a = reinterpret_cast<const __nv_bfloat162*>(&cur4), *b = reinterpret_cast<const __nv_bfloat162*>(&prev4);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 u = __bfloat1622float2(a[j]), v = __bfloat1622float2(b[j]);
            cur[2 * j] = u.x; cur[2 * j + 1] = u.y;
            step[2 * j] = v.x - u.x; step[2 * j + 1] = v.y - u.y;
        }
    }
    for (int s = 0; s < mixes; ++s) {
        const float4 m0 = *reinterpret_cast<const float4*>(mu + (int64_t)s * W + c), m1 = *reinterpret_cast<const float4*>(mu + (int64_t)s * W + c + 4);
        const float m[8] = {m0.x, m0.y, m0.z, m0.w, m1.x, m1.y, m1.z, m1.w};
        uint4 o;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int j = 0; j < 4; ++j)
            h[j] = __floats2bfloat162_rn(fmaf(step[2 * j], m[2 * j], cur[2 * j]), fmaf(step[2 * j + 1], m[2 * j + 1], cur[2 * j + 1]));
        *reinterpret_cast<uint4*>(out + s * plane + (int64_t)t * W + c) = o;
    }
}

enum DecayKind : int { kDoubleExp = 0, kRootedSigmoid = 1 };

// FAST (beside weights of 8 bits of mantissa): the hardware's exponential and logarithm, a few units in the last place of
// float32; float32 weights take the exact functions.
template <bool FAST>
__device__ __forceinline__ float decay_of(float v, int kind, float power) {
    if (kind == kDoubleExp) return FAST ? __expf(-__expf(v)) : expf(-expf(v));
    // sigmoid(v)^power = exp(power * log sigmoid(v)), log sigmoid(v) = min(v, 0) - log(1 + exp(-|v|))
    if constexpr (FAST) return __expf(power * (fminf(v, 0.0f) - __logf(1.0f + __expf(-fabsf(v)))));
    else return expf(power * (fminf(v, 0.0f) - log1pf(expf(-fabsf(v)))));
}

constexpr int kRankStep = 64;    // hidden entries staged at a time
constexpr int kDecayCols = 64;   // channels a block: a lane has two of them

// 4 warps: a lane is two channels, a warp TPW tokens at a time; a block walks `tiles` tiles of 4 TPW tokens with its channels'
// weights staged once (where the rank is at most kRankStep). wvec: rows of w may be read 16 bytes at a time.
template <typename TW, int TPW>
__global__ void __launch_bounds__(128) low_rank_decay_kernel(const float* __restrict__ z, int64_t ldz, const TW* __restrict__ w,
                                                             const float* __restrict__ bias, float* __restrict__ out, int Tn, int C, int R,
                                                             int hidden_tanh, int kind, float power, int tiles, int wvec) {
    __shared__ float ws[kRankStep][kDecayCols + 1];
    __shared__ __align__(16) float zs[4 * TPW][kRankStep];
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int c0 = blockIdx.x * kDecayCols;
    const float b0 = bias != nullptr && c0 + lane < C ? bias[c0 + lane] : 0.0f;
    const float b1 = bias != nullptr && c0 + lane + 32 < C ? bias[c0 + lane + 32] : 0.0f;
    bool waited = false;
    for (int tile = 0; tile < tiles; ++tile) {
        const int t0 = (blockIdx.y * tiles + tile) * (4 * TPW);
        if (t0 >= Tn) break;
        float acc[TPW][2];
#pragma unroll
        for (int i = 0; i < TPW; ++i) acc[i][0] = acc[i][1] = 0.0f;
        for (int r0 = 0; r0 < R; r0 += kRankStep) {
            __syncthreads();
            if (tile == 0 || R > kRankStep) {
                if (wvec) {
                    constexpr int N = 16 / sizeof(TW);
#pragma unroll
                    for (int e = threadIdx.x; e < kDecayCols * kRankStep / N; e += 128) {
                        const int c = e / (kRankStep / N), r = (e - c * (kRankStep / N)) * N;
                        uint4 raw = make_uint4(0u, 0u, 0u, 0u);
                        if (c0 + c < C && r0 + r < R) raw = *reinterpret_cast<const uint4*>(w + (int64_t)(c0 + c) * R + r0 + r);
                        const TW* v = reinterpret_cast<const TW*>(&raw);
#pragma unroll
                        for (int j = 0; j < N; ++j) ws[r + j][c] = to_f32(v[j]);
                    }
                } else {
                    for (int e = threadIdx.x; e < kDecayCols * kRankStep; e += 128) {
                        const int c = e / kRankStep, r = e - c * kRankStep;
                        ws[r][c] = c0 + c < C && r0 + r < R ? to_f32(w[(int64_t)(c0 + c) * R + r0 + r]) : 0.0f;
                    }
                }
            }
            if (!waited) {                             // (the weights depend on nothing)
                pdl_wait();
                waited = true;
            }
#pragma unroll 4
            for (int e = threadIdx.x; e < 4 * TPW * kRankStep; e += 128) {
                const int t = e / kRankStep, r = e - t * kRankStep;
                float v = t0 + t < Tn && r0 + r < R ? z[(int64_t)(t0 + t) * ldz + r0 + r] : 0.0f;
                if (hidden_tanh) v = tanhf(v);
                zs[t][r] = v;
            }
            __syncthreads();
            const int steps = min(kRankStep, R - r0);      // (entries from R on are zero: whole fours)
            for (int r = 0; r < steps; r += 4) {
                float u[4][2];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    u[j][0] = ws[r + j][lane];
                    u[j][1] = ws[r + j][lane + 32];
                }
#pragma unroll
                for (int i = 0; i < TPW; ++i) {
                    const float4 v = *reinterpret_cast<const float4*>(&zs[warp * TPW + i][r]);
                    const float vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        acc[i][0] = fmaf(u[j][0], vv[j], acc[i][0]);
                        acc[i][1] = fmaf(u[j][1], vv[j], acc[i][1]);
                    }
                }
            }
        }
        const int c = c0 + lane;
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const int t = t0 + warp * TPW + i;
            if (t >= Tn) break;
            if (c < C) out[(int64_t)t * C + c] = decay_of<sizeof(TW) == 2>(acc[i][0] + b0, kind, power);
            if (c + 32 < C) out[(int64_t)t * C + c + 32] = decay_of<sizeof(TW) == 2>(acc[i][1] + b1, kind, power);
        }
    }
}

}  // namespace

// x: [T, W] rows `ldx` apart; state: [*, W] in x's element type; mu: [mixes, W] float32; out: [mixes, T, W].
XS_API int xs_token_mix(const void* x, int64_t ldx, void* state, const float* mu, void* out, const int32_t* seq_of_token,
                        const int32_t* cu_seqlens, const int32_t* slots, int T, int W, int mixes, int dtype, cudaStream_t stream) {
    if (T == 0) return 0;
    XS_REQUIRE(T > 0 && W > 0 && ldx >= W && mixes > 0 && W <= 65535 * 128, "token_mix: %d tokens of %d, %d mixes", T, W, mixes);
    const int64_t plane = (int64_t)T * W;
    const uintptr_t all = (uintptr_t)x | (uintptr_t)state | (uintptr_t)mu | (uintptr_t)out;
    if (dtype == XS_BF16 && W % 8 == 0 && ldx % 8 == 0 && all % 16 == 0) {
        xs_launch(token_mix_vec_kernel, dim3(T, ceil_div_i(W, 8 * 128)), dim3(128), 0, stream, (const __nv_bfloat16*)x, ldx,
                  (__nv_bfloat16*)state, mu, (__nv_bfloat16*)out, seq_of_token, cu_seqlens, slots, plane, W, mixes);
        XS_LAUNCH_CHECK("token_mix");
        return 0;
    }
    XS_DISPATCH_DTYPE(dtype, TT,
                      xs_launch(token_mix_kernel<TT>, dim3(T, ceil_div_i(W, 128)), dim3(128), 0, stream, (const TT*)x, ldx, (TT*)state, mu,
                                (TT*)out, seq_of_token, cu_seqlens, slots, plane, W, mixes));
    XS_LAUNCH_CHECK("token_mix");
    return 0;
}

// z: [T, >= R] float32 rows `ldz` apart; w: [C, R] in the element type `w_dtype`; bias: [C] float32 or null; out: [T, C] float32.
// kind 0: exp(-exp(v)); 1: sigmoid(v)^power.
XS_API int xs_low_rank_decay(const float* z, int64_t ldz, const void* w, int w_dtype, const float* bias, float* out, int T, int C, int R,
                             int hidden_tanh, int kind, float power, cudaStream_t stream) {
    if (T == 0) return 0;
    XS_REQUIRE(T > 0 && C > 0 && R > 0 && ldz >= R && (kind == kDoubleExp || kind == kRootedSigmoid) && power > 0.0f,
               "low_rank_decay: %d tokens, %d channels, rank %d, kind %d", T, C, R, kind);
    XS_REQUIRE(T <= 65535 * 8, "low_rank_decay: %d tokens exceed the grid limit", T);
    const int cols = ceil_div_i(C, kDecayCols);
    const int wvec = (R * (w_dtype == XS_BF16 ? 2 : 4)) % 16 == 0 && (uintptr_t)w % 16 == 0;
    if (T >= 256) {
        const int all = ceil_div_i(T, 32);
        int tiles = ceil_div_i((int64_t)all * cols, 148 * 8);          // about one round of blocks
        if (tiles > 8) tiles = 8;
        XS_DISPATCH_DTYPE(w_dtype, TW,
                          xs_launch(low_rank_decay_kernel<TW, 8>, dim3(cols, ceil_div_i(all, tiles)), dim3(128), 0, stream, z, ldz,
                                    (const TW*)w, bias, out, T, C, R, hidden_tanh, kind, power, tiles, wvec));
    } else {
        XS_DISPATCH_DTYPE(w_dtype, TW,
                          xs_launch(low_rank_decay_kernel<TW, 2>, dim3(cols, ceil_div_i(T, 8)), dim3(128), 0, stream, z, ldz,
                                    (const TW*)w, bias, out, T, C, R, hidden_tanh, kind, power, 1, wvec));
    }
    XS_LAUNCH_CHECK("low_rank_decay");
    return 0;
}
