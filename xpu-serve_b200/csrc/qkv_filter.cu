// What stands between an attention layer's stacked q / k / v product and its attention when the projections are filtered over
// time and normed as a whole, in one pass over the product's rows:
//
//   u[t, c]  = x[t, c] + bias[c]                                    (a sequence's rows only: zeros before its first token)
//   f[t, c]  = sum_b taps[c, n - 1 - b] u[t - b, c]                 c over the q, k and v channels
//   q, k     = f / sqrt(sum over all q (k) channels of f^2 / count + eps) * w, then rotated head by head
//   q to its own tensor, k and v (as filtered) into the cache's pages
//
// `count` is the number of channels the norm is over in the checkpoint (heads that the kernels hold padded add zeros to the
// sum). The product's rows before a step come from the sequence's state [n - 1, C] (as the product left them, without the
// bias), which then moves on. A block a token: filtered values go to shared memory as float32 beside the two sums of squares,
// and are normed and rotated from there. All sums are float32 in an order that depends on the sizes alone.
#include "common.cuh"

int xs_filter_state(const void* x, int64_t ldx, void* state, const int32_t* cu_seqlens, const int32_t* slots, int n_seqs, int C,
                    int taps, int dtype, cudaStream_t stream);

namespace {

constexpr int kMaxFilterTaps = 16;

struct QkvFilterArgs {
    const void* x;               // [T, >= C] rows `ld` apart: q [Hq * D] | k [Hkv * D] | v [Hkv * DV]
    int64_t ld;
    const float* bias;           // [C] or null
    const float* taps;           // [n, C]: row b is the tap that looks b tokens back
    void* state;                 // [*, n - 1, C] or null (n == 1)
    void* q_out;                 // [T, Hq, D]
    void* pool;                  // pages: keys [Hkv, page, D], then values [Hkv, page, DV]
    const int32_t* page_table;
    const int32_t* seq_of_token;
    const int32_t* positions;
    const int32_t* cu_seqlens;
    const int32_t* slots;
    const float* q_w;            // [Hq * D] and [Hkv * D], or null: no norm
    const float* k_w;
    const float2* rope;          // [positions, D / 2] (cos, sin), or null
    int P, Hq, Hkv, D, DV, page_size, n, move_state;
    float q_count, k_count, eps;
};

// V neighbouring channels at a time
template <typename T, int V>
struct Chans;
template <typename T>
struct Chans<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f32(p[0]); }
    static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { p[0] = from_f32<T>(v[0]); }
};
template <>
struct Chans<float, 4> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 r = *reinterpret_cast<const float4*>(p);
        v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <>
struct Chans<__nv_bfloat16, 4> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
        const uint2 r = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
        const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
        v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
        uint2 r;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&r);
        h[0] = __floats2bfloat162_rn(v[0], v[1]);
        h[1] = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = r;
    }
};

// TAPS 0: any number up to kMaxFilterTaps.
template <typename T, int V, int TAPS>
__global__ void qkv_filter_kernel(const QkvFilterArgs a) {
    extern __shared__ __align__(16) float f_sm[];        // [q and k channels]
    __shared__ float red[2][32];
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int seq = a.seq_of_token[t], pos = a.positions[t];
    const int local = t - a.cu_seqlens[seq];
    const int64_t slot = a.slots[seq];
    const int nq = a.Hq * a.D, nk = a.Hkv * a.D, C = nq + nk + a.Hkv * a.DV;
    const int page = a.page_table[(int64_t)seq * a.P + pos / a.page_size], at = pos % a.page_size;
    T* kpage = (T*)a.pool + (int64_t)page * a.Hkv * a.page_size * (a.D + a.DV);
    T* vpage = kpage + (int64_t)a.Hkv * a.page_size * a.D;
    T* state = (T*)a.state + slot * (a.n - 1) * C;
    const T* x = (const T*)a.x;
    const int n = TAPS > 0 ? TAPS : a.n;
    constexpr int MOST = TAPS > 0 ? TAPS : kMaxFilterTaps;
    pdl_wait();
    float ssq = 0.0f, ssk = 0.0f;
    for (int c = threadIdx.x * V; c < C; c += blockDim.x * V) {
        float row[MOST][V];
#pragma unroll
        for (int b = 0; b < MOST; ++b) {
#pragma unroll
            for (int i = 0; i < V; ++i) row[b][i] = 0.0f;
            if (b < n && pos - b >= 0) {
                if (local - b >= 0) Chans<T, V>::load(x + (int64_t)(t - b) * a.ld + c, row[b]);
                else Chans<T, V>::load(state + (int64_t)(n - 1 - (b - local)) * C + c, row[b]);
            }
        }
        float bias[V], f[V];
#pragma unroll
        for (int i = 0; i < V; ++i) bias[i] = f[i] = 0.0f;
        if (a.bias != nullptr) Chans<float, V>::load(a.bias + c, bias);
#pragma unroll
        for (int b = MOST - 1; b >= 0; --b) {
            if (b < n) {
                float w[V];
                Chans<float, V>::load(a.taps + (int64_t)b * C + c, w);
#pragma unroll
                for (int i = 0; i < V; ++i) f[i] = fmaf(w[i], pos - b >= 0 ? row[b][i] + bias[i] : 0.0f, f[i]);
                // a step of one token a sequence: the row b before this token is b + 1 before the next (all were read above)
                if (a.move_state && b < n - 1) Chans<T, V>::store(state + (int64_t)(n - 2 - b) * C + c, row[b]);
            }
        }
        if (c < nq + nk) {
            float ss = 0.0f;
#pragma unroll
            for (int i = 0; i < V; ++i) ss = fmaf(f[i], f[i], ss);
            if (c < nq) ssq += ss;
            else ssk += ss;
            Chans<float, V>::store(f_sm + c, f);
        } else {
            const int vc = c - nq - nk;
            Chans<T, V>::store(vpage + ((int64_t)(vc / a.DV) * a.page_size + at) * a.DV + vc % a.DV, f);
        }
    }
    {
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
        ssq = warp_sum(ssq);
        ssk = warp_sum(ssk);
        if (lane == 0) {
            red[0][warp] = ssq;
            red[1][warp] = ssk;
        }
        __syncthreads();                                  // (the filtered values are in shared memory too)
        ssq = warp_sum(lane < warps ? red[0][lane] : 0.0f);
        ssk = warp_sum(lane < warps ? red[1][lane] : 0.0f);
    }
    const float iq = a.q_w != nullptr ? 1.0f / sqrtf(ssq / a.q_count + a.eps) : 1.0f;
    const float ik = a.k_w != nullptr ? 1.0f / sqrtf(ssk / a.k_count + a.eps) : 1.0f;
    const int half = a.D >> 1;
    const float2* cs = a.rope != nullptr ? a.rope + (int64_t)pos * half : nullptr;
    // pairs (i, i + D / 2) of every q and k head, V neighbouring pairs a thread
    const int pairs = (nq + nk) >> 1;
    for (int e = threadIdx.x * V; e < pairs; e += blockDim.x * V) {
        const int h = e / half, i = e - h * half;
        const int lo = h * a.D + i, hi = lo + half;
        float u[V], v[V];
        Chans<float, V>::load(f_sm + lo, u);
        Chans<float, V>::load(f_sm + hi, v);
        const bool is_q = h < a.Hq;
        const float* w = is_q ? a.q_w : a.k_w;
        if (w != nullptr) {
            const float inv = is_q ? iq : ik;
            float wu[V], wv[V];
            Chans<float, V>::load(w + (is_q ? lo : lo - nq), wu);
            Chans<float, V>::load(w + (is_q ? hi : hi - nq), wv);
#pragma unroll
            for (int j = 0; j < V; ++j) {
                u[j] = u[j] * inv * wu[j];
                v[j] = v[j] * inv * wv[j];
            }
        }
        if (cs != nullptr) {
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const float2 r = cs[i + j];
                const float a0 = u[j] * r.x - v[j] * r.y, a1 = v[j] * r.x + u[j] * r.y;
                u[j] = a0;
                v[j] = a1;
            }
        }
        T* dst = is_q ? (T*)a.q_out + (int64_t)t * nq + lo : kpage + ((int64_t)(h - a.Hq) * a.page_size + at) * a.D + i;
        Chans<T, V>::store(dst, u);
        Chans<T, V>::store(dst + half, v);
    }
}

// The same for long steps, kTile tokens a block: a channel's taps, bias and norm weights and the rows that neighbouring tokens
// share are read once for all of them. Only what a sequence's first TAPS - 1 tokens of the step look back to comes from its state.
constexpr int kTile = 4;

template <typename T, int TAPS>
__global__ void __launch_bounds__(256, 3) qkv_filter_tile_kernel(const QkvFilterArgs a, int n_tokens) {
    constexpr int V = 4, ROWS = kTile + TAPS - 1;
    extern __shared__ __align__(16) float f_sm[];        // [kTile][q and k channels]
    __shared__ float red[2 * kTile][16];
    pdl_launch_dependents();
    const int t0 = blockIdx.x * kTile;
    const int nq = a.Hq * a.D, nk = a.Hkv * a.D, C = nq + nk + a.Hkv * a.DV;
    int pos[kTile], local[kTile], seq[kTile];
    T* kpage[kTile];
#pragma unroll
    for (int i = 0; i < kTile; ++i) {
        const int t = min(t0 + i, n_tokens - 1);
        seq[i] = a.seq_of_token[t];
        pos[i] = a.positions[t];
    }
#pragma unroll
    for (int i = 0; i < kTile; ++i) {
        local[i] = min(t0 + i, n_tokens - 1) - a.cu_seqlens[seq[i]];
        const int page = a.page_table[(int64_t)seq[i] * a.P + pos[i] / a.page_size];
        kpage[i] = (T*)a.pool + (int64_t)page * a.Hkv * a.page_size * (a.D + a.DV);
    }
    const T* x = (const T*)a.x;
    pdl_wait();
    float ssq[kTile], ssk[kTile];
#pragma unroll
    for (int i = 0; i < kTile; ++i) ssq[i] = ssk[i] = 0.0f;
    for (int c = threadIdx.x * V; c < C; c += blockDim.x * V) {
        float rows[ROWS][V], w[TAPS][V], bias[V];
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {                  // row r is token t0 - (TAPS - 1) + r
            const int t = t0 - (TAPS - 1) + r;
#pragma unroll
            for (int v = 0; v < V; ++v) rows[r][v] = 0.0f;
            if (t >= 0 && t < n_tokens) Chans<T, V>::load(x + (int64_t)t * a.ld + c, rows[r]);
        }
#pragma unroll
        for (int b = 0; b < TAPS; ++b) Chans<float, V>::load(a.taps + (int64_t)b * C + c, w[b]);
#pragma unroll
        for (int v = 0; v < V; ++v) bias[v] = 0.0f;
        if (a.bias != nullptr) Chans<float, V>::load(a.bias + c, bias);
#pragma unroll
        for (int i = 0; i < kTile; ++i) {
            if (t0 + i >= n_tokens) break;
            float f[V];
#pragma unroll
            for (int v = 0; v < V; ++v) f[v] = 0.0f;
#pragma unroll
            for (int b = TAPS - 1; b >= 0; --b) {
                if (pos[i] - b < 0) continue;             // before the sequence: zeros
                if (local[i] - b >= 0) {
#pragma unroll
                    for (int v = 0; v < V; ++v) f[v] = fmaf(w[b][v], rows[i + TAPS - 1 - b][v] + bias[v], f[v]);
                } else {
                    float sv[V];
                    Chans<T, V>::load((const T*)a.state + ((int64_t)a.slots[seq[i]] * (TAPS - 1) + (TAPS - 1 - (b - local[i]))) * C + c, sv);
#pragma unroll
                    for (int v = 0; v < V; ++v) f[v] = fmaf(w[b][v], sv[v] + bias[v], f[v]);
                }
            }
            if (c < nq + nk) {
                float ss = 0.0f;
#pragma unroll
                for (int v = 0; v < V; ++v) ss = fmaf(f[v], f[v], ss);
                if (c < nq) ssq[i] += ss;
                else ssk[i] += ss;
                Chans<float, V>::store(f_sm + i * (nq + nk) + c, f);
            } else {
                const int vc = c - nq - nk, vh = vc / a.DV;
                Chans<T, V>::store(kpage[i] + (int64_t)a.Hkv * a.page_size * a.D + ((int64_t)vh * a.page_size + pos[i] % a.page_size) * a.DV + (vc - vh * a.DV), f);
            }
        }
    }
    {
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
#pragma unroll
        for (int i = 0; i < kTile; ++i) {
            ssq[i] = warp_sum(ssq[i]);
            ssk[i] = warp_sum(ssk[i]);
            if (lane == 0) {
                red[2 * i][warp] = ssq[i];
                red[2 * i + 1][warp] = ssk[i];
            }
        }
        __syncthreads();                                  // (the filtered values are in shared memory too)
#pragma unroll
        for (int i = 0; i < kTile; ++i) {
            ssq[i] = warp_sum(lane < warps ? red[2 * i][lane] : 0.0f);
            ssk[i] = warp_sum(lane < warps ? red[2 * i + 1][lane] : 0.0f);
        }
    }
    const int half = a.D >> 1, pairs = (nq + nk) >> 1;
    for (int e = threadIdx.x * V; e < pairs; e += blockDim.x * V) {
        const int h = e / half, p = e - h * half;
        const int lo = h * a.D + p, hi = lo + half;
        const bool is_q = h < a.Hq;
        const float* wt = is_q ? a.q_w : a.k_w;
        float wu[V], wv[V];
#pragma unroll
        for (int v = 0; v < V; ++v) wu[v] = wv[v] = 1.0f;
        if (wt != nullptr) {
            Chans<float, V>::load(wt + (is_q ? lo : lo - nq), wu);
            Chans<float, V>::load(wt + (is_q ? hi : hi - nq), wv);
        }
#pragma unroll
        for (int i = 0; i < kTile; ++i) {
            if (t0 + i >= n_tokens) break;
            float y[V], z[V];
            Chans<float, V>::load(f_sm + i * (nq + nk) + lo, y);
            Chans<float, V>::load(f_sm + i * (nq + nk) + hi, z);
            if (wt != nullptr) {
                const float inv = is_q ? 1.0f / sqrtf(ssq[i] / a.q_count + a.eps) : 1.0f / sqrtf(ssk[i] / a.k_count + a.eps);
#pragma unroll
                for (int v = 0; v < V; ++v) {
                    y[v] = y[v] * inv * wu[v];
                    z[v] = z[v] * inv * wv[v];
                }
            }
            if (a.rope != nullptr) {
                const float4* cs = reinterpret_cast<const float4*>(a.rope + (int64_t)pos[i] * half + p);
                const float4 c0 = cs[0], c1 = cs[1];
                const float co[V] = {c0.x, c0.z, c1.x, c1.z}, si[V] = {c0.y, c0.w, c1.y, c1.w};
#pragma unroll
                for (int v = 0; v < V; ++v) {
                    const float a0 = y[v] * co[v] - z[v] * si[v], a1 = z[v] * co[v] + y[v] * si[v];
                    y[v] = a0;
                    z[v] = a1;
                }
            }
            T* dst = is_q ? (T*)a.q_out + (int64_t)(t0 + i) * nq + lo : kpage[i] + ((int64_t)(h - a.Hq) * a.page_size + pos[i] % a.page_size) * a.D + p;
            Chans<T, V>::store(dst, y);
            Chans<T, V>::store(dst + half, z);
        }
    }
}

template <typename T, int TAPS>
void launch_tile(const QkvFilterArgs& a, int Tn, cudaStream_t stream) {
    const int groups = ceil_div_i(a.Hq * a.D + a.Hkv * (a.D + a.DV), 4);
    const int rounds = ceil_div_i(groups, 256);
    const int threads = ceil_div_i(ceil_div_i(groups, rounds), 32) * 32;      // every thread the same number of channels, but for the last warp's
    const size_t smem = (size_t)kTile * (a.Hq + a.Hkv) * a.D * sizeof(float);
    if (smem > 40 * 1024)
        cudaFuncSetAttribute(qkv_filter_tile_kernel<T, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    xs_launch(qkv_filter_tile_kernel<T, TAPS>, dim3(ceil_div_i(Tn, kTile)), dim3(threads), smem, stream, a, Tn);
}

template <typename T>
int launch_filter(const QkvFilterArgs& a, int Tn, bool vec, cudaStream_t stream) {
    const int C = a.Hq * a.D + a.Hkv * (a.D + a.DV);
    const size_t smem = (size_t)(a.Hq + a.Hkv) * a.D * sizeof(float);
    const int work = vec ? ceil_div_i(C, 4) : C;
    const int threads = work >= 512 ? 512 : work >= 256 ? 256 : 128;
    if (vec && !a.move_state && Tn >= 256 && a.n <= 5 && smem * kTile <= 160 * 1024 && (uintptr_t)a.rope % 16 == 0) {
        if (a.n == 1) launch_tile<T, 1>(a, Tn, stream);
        else if (a.n == 2) launch_tile<T, 2>(a, Tn, stream);
        else if (a.n == 3) launch_tile<T, 3>(a, Tn, stream);
        else if (a.n == 4) launch_tile<T, 4>(a, Tn, stream);
        else launch_tile<T, 5>(a, Tn, stream);
        return 0;
    }
#define XS_GO2(V, N)                                                                                                       \
    do {                                                                                                                   \
        if (smem > 47 * 1024)                                                                                              \
            cudaFuncSetAttribute(qkv_filter_kernel<T, V, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);      \
        xs_launch(qkv_filter_kernel<T, V, N>, dim3(Tn), dim3(threads), smem, stream, a);                                   \
    } while (0)
    if (!vec) XS_GO2(1, 0);
    else if (a.n == 1) XS_GO2(4, 1);
    else if (a.n == 2) XS_GO2(4, 2);
    else if (a.n == 3) XS_GO2(4, 3);
    else if (a.n == 4) XS_GO2(4, 4);
    else if (a.n <= 8) XS_GO2(4, 0);
    else XS_GO2(1, 0);
#undef XS_GO2
    return 0;
}

}  // namespace

// all_single: every sequence brings one token (the kernel then moves the state on itself; otherwise a second one does).
XS_API int xs_qkv_filter(const void* x, int64_t ld, const float* bias, const float* taps, void* state, void* q_out, void* pool,
                         const int32_t* page_table, int P, const int32_t* seq_of_token, const int32_t* positions,
                         const int32_t* cu_seqlens, const int32_t* slots, const float* q_w, const float* k_w, const float* rope,
                         int T, int n_seqs, int Hq, int Hkv, int D, int DV, int n_taps, int q_count, int k_count, int page_size,
                         float eps, int all_single, int dtype, cudaStream_t stream) {
    if (T == 0) return 0;
    XS_REQUIRE(T > 0 && n_seqs > 0 && Hq > 0 && Hkv > 0 && Hq % Hkv == 0 && D > 0 && D % 2 == 0 && DV > 0 && page_size > 0 && P > 0,
               "qkv_filter: %d tokens, %d heads over %d, sizes %d / %d", T, Hq, Hkv, D, DV);
    XS_REQUIRE(n_taps >= 1 && n_taps <= kMaxFilterTaps && (n_taps == 1 || state != nullptr), "qkv_filter: %d taps (1 to %d)", n_taps, kMaxFilterTaps);
    XS_REQUIRE(!all_single || T == n_seqs, "qkv_filter: %d tokens for %d sequences of one token each", T, n_seqs);
    const int C = Hq * D + Hkv * (D + DV);
    XS_REQUIRE(ld >= C && q_count > 0 && k_count > 0, "qkv_filter: rows %lld apart for %d channels", (long long)ld, C);
    XS_REQUIRE((size_t)(Hq + Hkv) * D * 4 <= 200 * 1024, "qkv_filter: %d + %d heads of %d do not fit shared memory", Hq, Hkv, D);
    QkvFilterArgs a{x, ld, bias, taps, state, q_out, pool, page_table, seq_of_token, positions, cu_seqlens, slots, q_w, k_w,
                    (const float2*)rope, P, Hq, Hkv, D, DV, page_size, n_taps, all_single && n_taps > 1 ? 1 : 0,
                    (float)q_count, (float)k_count, eps};
    const uintptr_t all = (uintptr_t)x | (uintptr_t)bias | (uintptr_t)taps | (uintptr_t)state | (uintptr_t)q_out | (uintptr_t)pool |
                          (uintptr_t)q_w | (uintptr_t)k_w;
    const bool vec = D % 8 == 0 && DV % 4 == 0 && ld % 4 == 0 && all % 16 == 0;
    XS_DISPATCH_DTYPE(dtype, TT, launch_filter<TT>(a, T, vec, stream));
    XS_LAUNCH_CHECK("qkv_filter");
    if (n_taps > 1 && !all_single) return xs_filter_state(x, ld, state, cu_seqlens, slots, n_seqs, C, n_taps, dtype, stream);
    return 0;
}
