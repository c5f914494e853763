// PolyNorm: out = a N(z) + b N(z^2) + c N(z^3) + e over the rows of z [T, F], powers element by element and N(y) =
// y / sqrt(mean(y^2) + eps) over the row; coef holds (a, b, c, e). Sums and arithmetic in float32.
//
// One block a row: the row's values are read once (kept in registers where they fit, 16 bytes a load), the sums of z^2, z^4
// and z^6 meet across the block, and each output is ((c3 z + c2) z + c1) z + e with the three norms in the coefficients.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;
constexpr int kVecs = 4;          // 16-byte pieces a thread keeps: rows of up to 256 * 4 * 8 = 8,192 values

// The block's three sums; every thread gets them (`sm` holds 3 * 32 floats).
__device__ __forceinline__ float3 block_sum3(float a, float b, float c, float* sm) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    c = warp_sum(c);
    if (lane == 0) {
        sm[warp] = a;
        sm[32 + warp] = b;
        sm[64 + warp] = c;
    }
    __syncthreads();
    return make_float3(warp_sum(lane < warps ? sm[lane] : 0.0f), warp_sum(lane < warps ? sm[32 + lane] : 0.0f),
                       warp_sum(lane < warps ? sm[64 + lane] : 0.0f));
}

struct PolyCoef {
    float c1, c2, c3, e;
    __device__ __forceinline__ float operator()(float z) const { return fmaf(fmaf(fmaf(c3, z, c2), z, c1), z, e); }
};

__device__ __forceinline__ PolyCoef poly_coef(float3 s, const float* coef, int F, float eps) {
    const float n = (float)F;
    return {coef[0] / sqrtf(s.x / n + eps), coef[1] / sqrtf(s.y / n + eps), coef[2] / sqrtf(s.z / n + eps), coef[3]};
}

template <typename T>
__global__ void __launch_bounds__(kThreads) poly_norm_kernel(const T* __restrict__ z, int64_t ldz, const float* __restrict__ coef,
                                                             T* __restrict__ out, int F, float eps) {
    __shared__ float sm[96];
    pdl_launch_dependents();
    pdl_wait();
    const T* row = z + (int64_t)blockIdx.x * ldz;
    float s2 = 0.0f, s4 = 0.0f, s6 = 0.0f;
    for (int i = threadIdx.x; i < F; i += kThreads) {
        const float v = to_f32(row[i]), q = v * v;
        s2 += q;
        s4 = fmaf(q, q, s4);
        s6 = fmaf(q * q, q, s6);
    }
    const PolyCoef p = poly_coef(block_sum3(s2, s4, s6, sm), coef, F, eps);
    for (int i = threadIdx.x; i < F; i += kThreads) out[(int64_t)blockIdx.x * F + i] = from_f32<T>(p(to_f32(row[i])));
}

__global__ void __launch_bounds__(kThreads) poly_norm_vec_kernel(const __nv_bfloat16* __restrict__ z, int64_t ldz, const float* __restrict__ coef,
                                                                 __nv_bfloat16* __restrict__ out, int F8, float eps) {
    __shared__ float sm[96];
    pdl_launch_dependents();
    pdl_wait();
    const uint4* row = reinterpret_cast<const uint4*>(z + (int64_t)blockIdx.x * ldz);
    uint4 raw[kVecs];
#pragma unroll
    for (int k = 0; k < kVecs; ++k) {
        const int i = threadIdx.x + k * kThreads;
        raw[k] = i < F8 ? row[i] : make_uint4(0u, 0u, 0u, 0u);
    }
    float s2 = 0.0f, s4 = 0.0f, s6 = 0.0f;
#pragma unroll
    for (int k = 0; k < kVecs; ++k) {
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw[k]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 f = __bfloat1622float2(h2[j]);
            const float q0 = f.x * f.x, q1 = f.y * f.y;
            s2 += q0 + q1;
            s4 = fmaf(q0, q0, fmaf(q1, q1, s4));
            s6 = fmaf(q0 * q0, q0, fmaf(q1 * q1, q1, s6));
        }
    }
    const PolyCoef p = poly_coef(block_sum3(s2, s4, s6, sm), coef, F8 * 8, eps);
    uint4* dst = reinterpret_cast<uint4*>(out) + (int64_t)blockIdx.x * F8;
#pragma unroll
    for (int k = 0; k < kVecs; ++k) {
        const int i = threadIdx.x + k * kThreads;
        if (i >= F8) break;
        __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&raw[k]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 f = __bfloat1622float2(h2[j]);
            h2[j] = __floats2bfloat162_rn(p(f.x), p(f.y));
        }
        dst[i] = raw[k];
    }
}

}  // namespace

XS_API int xs_poly_norm(const void* z, int64_t ldz, const float* coef, void* out, int T, int F, float eps, int dtype,
                        cudaStream_t stream) {
    if (T == 0) return 0;
    XS_REQUIRE(T > 0 && F > 0 && ldz >= F && coef != nullptr, "poly_norm: %d rows of %d (stride %lld)", T, F, (long long)ldz);
    if (dtype == XS_BF16 && F % 8 == 0 && F <= kThreads * kVecs * 8 && ldz % 8 == 0 && (uintptr_t)z % 16 == 0 && (uintptr_t)out % 16 == 0) {
        xs_launch(poly_norm_vec_kernel, dim3(T), dim3(kThreads), 0, stream, (const __nv_bfloat16*)z, ldz, coef, (__nv_bfloat16*)out, F / 8, eps);
        XS_LAUNCH_CHECK("poly_norm");
        return 0;
    }
    XS_DISPATCH_DTYPE(dtype, TT,
                      xs_launch(poly_norm_kernel<TT>, dim3(T), dim3(kThreads), 0, stream, (const TT*)z, ldz, coef, (TT*)out, F, eps));
    XS_LAUNCH_CHECK("poly_norm");
    return 0;
}
