// The kernels of attention_mma.cu as templates over the head sizes: keys of D and values of DV channels, prompts
// (attention_mma_kernel) and single tokens (attention_decode_mma_kernel), and what launches them. attention_mma.cu has the
// equal sizes and the interface, attention_pairs.cu the unequal ones.
#pragma once

#include <cuda.h>

#include "common.cuh"
#include "tc_common.cuh"

namespace xs_attn {

extern int g_attn_decode_stages;
int sm_count();

constexpr int BM = 64;       // query rows per CTA
constexpr int BN = 64;       // keys per block = page size
constexpr int NTHREADS = 128;

struct AttnParams {
    const __nv_bfloat16* q;          // [T, Hq, D]
    const __nv_bfloat16* pool;       // pages: keys [Hkv, 64, D], then (planes 2) values [Hkv, 64, DV]
    const int32_t* page_table;       // [n_seqs, P]
    int P;
    const int32_t* cu_seqlens;       // [n_seqs + 1]
    const int32_t* kv_lens;          // [n_seqs] length after this step
    const __nv_bfloat16* gate;       // [T, ld_gate] gate logits (one a head, or with gate_channels one a channel) or null
    int64_t ld_gate;
    __nv_bfloat16* out;              // [T, Hq, DV], tokens `ld_out` elements apart
    int64_t ld_out;
    float* part_o;                   // [T * Hq, splits, DV]
    float* part_ml;                  // [T * Hq, splits, 2]
    int Hq, Hkv, G, tokens_per_tile, window, splits;
    int keep;                        // beside a window: the sequence's first positions that stay visible
    int planes;                      // 1: the keys are the values too (DV == D), nothing is loaded for them
    int plus_one;                    // the softmax's denominator has one more term of score 0
    int gate_channels;
    int prefetch_blocks;             // decode: how many of a CTA's first key blocks are hinted into L2 before the wait
    int decode_rows;                 // every tile has at most 16 rows: the warps split the keys instead
    float scale_log2;
    float cap_in, cap_out;           // cap_out > 0: a score is cap_out * tanh(q.k * cap_in) (base-2 units) instead of q.k * scale_log2
    unsigned int* counters;          // decode with key splits: one zeroed word per (sequence, kv head), left zeroed; or null
};

// 1 / denominator of a row whose exponentials, relative to the maximum m (base 2), add up to l.
__device__ __forceinline__ float inv_denominator(float l, float m, int plus_one) {
    if (plus_one) l += exp2f(-m);         // (no key seen: m = -inf, the sum is infinite and the result 0)
    return l > 0.0f ? 1.0f / l : 0.0f;
}
__device__ __forceinline__ float gate_of(const AttnParams& p, int64_t t, int64_t at) {
    return 1.0f / (1.0f + __expf(-__bfloat162float(p.gate[t * p.ld_gate + at])));
}

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool valid) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = valid ? 16 : 0;   // 0: the 16 bytes are zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(bytes));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

__device__ __forceinline__ void ldmatrix_x4(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(s));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(s));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 2^x by the hardware approximation (2 ulp; -inf gives 0): the softmax weights are rounded to bfloat16 anyway
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// One page of keys and values of one kv head into shared memory; rows from `valid` on are zero.
template <int D, int DV>
__device__ __forceinline__ void load_kv_block(const AttnParams& p, int page, int kvh, int valid, bool own_v, __nv_bfloat16* ks,
                                              __nv_bfloat16* vs) {
    constexpr int CHUNKS = D / 8, VCHUNKS = DV / 8, LD = D + 8, LV = DV + 8;
    const __nv_bfloat16* base = p.pool + (int64_t)max(page, 0) * p.Hkv * BN * (own_v ? D + DV : D);
    const __nv_bfloat16* kbase = base + (int64_t)kvh * BN * D;
    const __nv_bfloat16* vbase = base + (int64_t)p.Hkv * BN * D + (int64_t)kvh * BN * DV;
    if (D == DV && own_v) {
        for (int c = threadIdx.x; c < BN * CHUNKS; c += NTHREADS) {
            const int r = c / CHUNKS, ch = c % CHUNKS;
            const bool ok = r < valid;
            cp_async16(ks + r * LD + ch * 8, kbase + (ok ? r * D + ch * 8 : 0), ok);
            cp_async16(vs + r * LV + ch * 8, vbase + (ok ? r * DV + ch * 8 : 0), ok);
        }
        return;
    }
    for (int c = threadIdx.x; c < BN * CHUNKS; c += NTHREADS) {
        const int r = c / CHUNKS, ch = c % CHUNKS;
        cp_async16(ks + r * LD + ch * 8, kbase + (r < valid ? r * D + ch * 8 : 0), r < valid);
    }
    if (!own_v) return;
    for (int c = threadIdx.x; c < BN * VCHUNKS; c += NTHREADS) {
        const int r = c / VCHUNKS, ch = c % VCHUNKS;
        cp_async16(vs + r * LV + ch * 8, vbase + (r < valid ? r * DV + ch * 8 : 0), r < valid);
    }
}

// CTAs an SM that the prompt kernel's registers are bounded for.
constexpr int prompt_ctas(int D, int DV) { return D + DV <= 128 ? 4 : D + DV <= 160 ? 3 : 2; }

template <int D, int DV, int NST>
__global__ void __launch_bounds__(NTHREADS, prompt_ctas(D, DV)) attention_mma_kernel(const AttnParams p) {
    constexpr int LD = D + 8;              // padded row: ldmatrix reads 8 rows without bank conflicts
    constexpr int LV = DV + 8;
    constexpr int KSTEPS = D / 16;         // k-steps of Q K^T
    constexpr int DTILES = DV / 8;         // n-tiles of the output
    constexpr int CHUNKS = D / 8;          // 16-byte chunks per row of queries and keys
    constexpr int VCHUNKS = DV / 8;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* q_sm = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* k_sm = q_sm + BM * LD;            // [NST][BN][LD]
    const bool own_v = DV != D || p.planes > 1;      // (else the keys' rows serve as the values')
    __nv_bfloat16* v_sm = own_v ? k_sm + NST * BN * LD : k_sm;      // [NST][BN][LV]

    pdl_launch_dependents();
    pdl_wait();
    // later tiles see more keys: they are started first, so that the short ones fill the tail
    const int tile = gridDim.x - 1 - blockIdx.x, seq = blockIdx.y;
    const int kvh = blockIdx.z / p.splits, split = blockIdx.z % p.splits;
    const int tok_begin = p.cu_seqlens[seq];
    const int q_len = p.cu_seqlens[seq + 1] - tok_begin;
    const int t0 = tile * p.tokens_per_tile;
    if (t0 >= q_len) return;
    const int nt = min(p.tokens_per_tile, q_len - t0);
    const int kv_len = p.kv_lens[seq];
    const int pos0 = kv_len - q_len + t0;
    const int hi = pos0 + nt;                                     // keys from hi on do not matter to this tile
    const XsBlocks blocks = xs_blocks(pos0, hi, p.window, p.keep, BN);
    const int bs = (int)((int64_t)blocks.count * split / p.splits);           // this CTA's share, as indices of `blocks`
    const int be = (int)((int64_t)blocks.count * (split + 1) / p.splits);
    const int32_t* table = p.page_table + (int64_t)seq * p.P;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int G = p.G;
    const int rows_valid = nt * G;
    const bool warp_active = warp * 16 < rows_valid;

    // ---- Q tile: row r = (token t0 + r / G, head kvh * G + r % G); invalid rows are zero
    for (int c = threadIdx.x; c < BM * CHUNKS; c += NTHREADS) {
        const int r = c / CHUNKS, ch = c % CHUNKS;
        const bool ok = r < rows_valid;
        const int ti = ok ? r / G : 0, g = ok ? r % G : 0;
        const __nv_bfloat16* src = p.q + ((int64_t)(tok_begin + t0 + ti) * p.Hq + kvh * G + g) * D + ch * 8;
        cp_async16(q_sm + r * LD + ch * 8, src, ok);
    }
    auto load_block = [&](int i, int stage) {
        const int b = blocks.at(i);
        const int page = table[b];             // a page given back (-1) is never read: its rows are zero-filled
        load_kv_block<D, DV>(p, page, kvh, page >= 0 ? hi - b * BN : 0, own_v, k_sm + stage * BN * LD, v_sm + stage * BN * LV);
    };
    // NST - 1 blocks are requested before the first is used; one commit group per block, empty ones too,
    // so that "all but the newest NST - 2 groups have landed" always means "block b is here"
#pragma unroll
    for (int s = 0; s < NST - 1; ++s) {
        if (bs + s < be) load_block(bs + s, s);
        cp_async_commit();
    }

    // this thread's two rows and their positions (-1: no key is visible)
    const int r1 = warp * 16 + (lane >> 2), r2 = r1 + 8;
    const int pos1 = r1 < rows_valid ? pos0 + r1 / G : -1;
    const int pos2 = r2 < rows_valid ? pos0 + r2 / G : -1;
    const int lo1 = xs_first_visible(pos1, p.window), lo2 = xs_first_visible(pos2, p.window);     // found once: may cost a division

    float o[DTILES][4];
#pragma unroll
    for (int i = 0; i < DTILES; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m1 = -INFINITY, m2 = -INFINITY, l1 = 0.0f, l2 = 0.0f;
    unsigned qf[KSTEPS][4];
    bool q_loaded = false;

    for (int i_blk = bs, it = 0; i_blk < be; ++i_blk, ++it) {
        const int stage = it % NST, b = blocks.at(i_blk);
        cp_async_wait<NST - 2>();
        __syncthreads();            // block b has landed for everyone, and everyone is done with block b - 1
        if (i_blk + NST - 1 < be) load_block(i_blk + NST - 1, (it + NST - 1) % NST);   // into the stage block b - 1 used
        cp_async_commit();
        if (warp_active) {
            if (!q_loaded) {
#pragma unroll
                for (int kk = 0; kk < KSTEPS; ++kk)
                    ldmatrix_x4(qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3],
                                q_sm + (warp * 16 + (lane & 15)) * LD + kk * 16 + (lane >> 4) * 8);
                q_loaded = true;
            }
            const __nv_bfloat16* ks = k_sm + stage * BN * LD;
            const __nv_bfloat16* vs = v_sm + stage * BN * LV;
            float s[BN / 8][4];
#pragma unroll
            for (int i = 0; i < BN / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
#pragma unroll
            for (int kk = 0; kk < KSTEPS; ++kk) {
#pragma unroll
                for (int np = 0; np < BN / 16; ++np) {
                    unsigned b0, b1, b2, b3;
                    ldmatrix_x4(b0, b1, b2, b3,
                                ks + (np * 16 + (lane >> 4) * 8 + (lane & 7)) * LD + kk * 16 + ((lane >> 3) & 1) * 8);
                    mma_bf16(s[2 * np], qf[kk], b0, b1);
                    mma_bf16(s[2 * np + 1], qf[kk], b2, b3);
                }
            }
            const float to_log2 = p.cap_out > 0.0f ? 1.0f : p.scale_log2;
            if (p.cap_out > 0.0f) xs_cap_scores<BN / 2>(&s[0][0], p.cap_in, p.cap_out);
            // scale, mask, running max. A block that every row of the tile sees whole (all of it at or before
            // the tile's first position and inside every row's window) needs no per-element test.
            const int key0 = b * BN + (lane & 3) * 2;
            const bool whole = b * BN + BN - 1 <= pos0 && (b * BN >= xs_first_visible(pos0 + nt - 1, p.window) || b * BN + BN <= p.keep);
            float mx1 = -INFINITY, mx2 = -INFINITY;
            if (whole) {
#pragma unroll
                for (int i = 0; i < BN / 8; ++i) {
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        s[i][e] = pos1 >= 0 ? s[i][e] * to_log2 : -INFINITY;
                        s[i][2 + e] = pos2 >= 0 ? s[i][2 + e] * to_log2 : -INFINITY;
                        mx1 = fmaxf(mx1, s[i][e]);
                        mx2 = fmaxf(mx2, s[i][2 + e]);
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < BN / 8; ++i) {
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int key = key0 + i * 8 + e;
                        const bool v1 = key <= pos1 && (key >= lo1 || key < p.keep);
                        const bool v2 = key <= pos2 && (key >= lo2 || key < p.keep);
                        s[i][e] = v1 ? s[i][e] * to_log2 : -INFINITY;
                        s[i][2 + e] = v2 ? s[i][2 + e] * to_log2 : -INFINITY;
                        mx1 = fmaxf(mx1, s[i][e]);
                        mx2 = fmaxf(mx2, s[i][2 + e]);
                    }
                }
            }
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
            mx2 = fmaxf(mx2, __shfl_xor_sync(0xffffffffu, mx2, 1));
            mx2 = fmaxf(mx2, __shfl_xor_sync(0xffffffffu, mx2, 2));
            const float mn1 = fmaxf(m1, mx1), mn2 = fmaxf(m2, mx2);
            const float base1 = mn1 == -INFINITY ? 0.0f : mn1, base2 = mn2 == -INFINITY ? 0.0f : mn2;
            const float c1 = fast_exp2(m1 - base1), c2 = fast_exp2(m2 - base2);   // 0 while nothing was seen
            m1 = mn1;
            m2 = mn2;
            l1 *= c1;
            l2 *= c2;
#pragma unroll
            for (int i = 0; i < DTILES; ++i) {
                o[i][0] *= c1;
                o[i][1] *= c1;
                o[i][2] *= c2;
                o[i][3] *= c2;
            }
            unsigned pf[BN / 16][4];
#pragma unroll
            for (int i = 0; i < BN / 8; ++i) {
                const float p0 = fast_exp2(s[i][0] - base1), p1 = fast_exp2(s[i][1] - base1);
                const float p2 = fast_exp2(s[i][2] - base2), p3 = fast_exp2(s[i][3] - base2);
                l1 += p0 + p1;
                l2 += p2 + p3;
                pf[i >> 1][(i & 1) * 2 + 0] = pack_bf16(p0, p1);
                pf[i >> 1][(i & 1) * 2 + 1] = pack_bf16(p2, p3);
            }
#pragma unroll
            for (int kk = 0; kk < BN / 16; ++kk) {
#pragma unroll
                for (int dp = 0; dp < DV / 16; ++dp) {
                    unsigned b0, b1, b2, b3;
                    ldmatrix_x4_trans(b0, b1, b2, b3,
                                      vs + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LV + dp * 16 + (lane >> 4) * 8);
                    mma_bf16(o[2 * dp], pf[kk], b0, b1);
                    mma_bf16(o[2 * dp + 1], pf[kk], b2, b3);
                }
            }
        }
    }
    cp_async_wait<0>();
    if (!warp_active) return;

    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    l2 += __shfl_xor_sync(0xffffffffu, l2, 1);
    l2 += __shfl_xor_sync(0xffffffffu, l2, 2);

#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = half == 0 ? r1 : r2;
        if (r >= rows_valid) continue;
        const int t = tok_begin + t0 + r / G, h = kvh * G + r % G;
        const float l = half == 0 ? l1 : l2, m = half == 0 ? m1 : m2;
        const int64_t row = (int64_t)t * p.Hq + h;
        if (p.splits == 1) {
            float f = inv_denominator(l, m, p.plus_one);
            if (p.gate != nullptr && !p.gate_channels) f *= gate_of(p, t, h);
            __nv_bfloat16* dst = p.out + (int64_t)t * p.ld_out + h * DV + (lane & 3) * 2;
            __nv_bfloat162 gates[DTILES];        // (all asked for before the first is used)
            if (p.gate_channels) {
                const __nv_bfloat16* from = p.gate + (int64_t)t * p.ld_gate + h * DV + (lane & 3) * 2;
#pragma unroll
                for (int i = 0; i < DTILES; ++i) gates[i] = *reinterpret_cast<const __nv_bfloat162*>(from + i * 8);
            }
#pragma unroll
            for (int i = 0; i < DTILES; ++i) {
                float g0 = f, g1 = f;
                if (p.gate_channels) {
                    const float2 z = __bfloat1622float2(gates[i]);
                    g0 = __fdividef(f, 1.0f + __expf(-z.x));
                    g1 = __fdividef(f, 1.0f + __expf(-z.y));
                }
                *reinterpret_cast<__nv_bfloat162*>(dst + i * 8) =
                    __floats2bfloat162_rn(o[i][half * 2] * g0, o[i][half * 2 + 1] * g1);
            }
        } else {
            float* dst = p.part_o + (row * p.splits + split) * DV + (lane & 3) * 2;
#pragma unroll
            for (int i = 0; i < DTILES; ++i)
                *reinterpret_cast<float2*>(dst + i * 8) = make_float2(o[i][half * 2], o[i][half * 2 + 1]);
            if ((lane & 3) == 0) {
                p.part_ml[(row * p.splits + split) * 2 + 0] = m;
                p.part_ml[(row * p.splits + split) * 2 + 1] = l;
            }
        }
    }
}

// Decoding (at most 16 query rows a tile: one token's group of heads): the rows would keep a single warp
// busy, so here the four warps split every 64-key block instead, 16 keys each, each with its own
// running maximum, sum and output; they are merged through shared memory at the end. Everything else
// (paging, masks, splits, zero-filled tails) is as in the kernel above.
template <int D, int DV, int NST>
__global__ void __launch_bounds__(NTHREADS) attention_decode_mma_kernel(const AttnParams p) {
    constexpr int LD = D + 8;
    constexpr int LV = DV + 8;
    constexpr int KSTEPS = D / 16;
    constexpr int DTILES = DV / 8;
    constexpr int CHUNKS = D / 8;
    constexpr int VCHUNKS = DV / 8;
    constexpr int QROWS = 16;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* q_sm = reinterpret_cast<__nv_bfloat16*>(smem_raw);    // [16][LD]
    __nv_bfloat16* k_sm = q_sm + QROWS * LD;                             // [NST][BN][LD]
    const bool own_v = DV != D || p.planes > 1;
    __nv_bfloat16* v_sm = own_v ? k_sm + NST * BN * LD : k_sm;           // [NST][BN][LV]
    __shared__ float sm_m[4][QROWS], sm_l[4][QROWS];
    __shared__ int pages_sm[64];

    pdl_launch_dependents();
    // The step's description (lengths, page table) was copied to the device before the step began, and cached
    // keys and values of earlier positions do not change during a step: the first blocks of this CTA's share of
    // the cache are asked into L2 before waiting for the kernel that writes the current position's keys and
    // values. Only the first: hints for a whole long share (hundreds of MB over all CTAs) push one another out of
    // L2 and the cache is then read from memory twice (64 sequences of 1k to 24k keys: 483 us with the whole share
    // hinted, 308 us with two blocks).
    const int seq = blockIdx.y;
    const int kvh = blockIdx.z / p.splits, split = blockIdx.z % p.splits;
    const int tok_begin = p.cu_seqlens[seq];
    const int q_len = p.cu_seqlens[seq + 1] - tok_begin;
    const int t0 = blockIdx.x * p.tokens_per_tile;
    if (t0 >= q_len) return;
    const int nt = min(p.tokens_per_tile, q_len - t0);
    const int kv_len = p.kv_lens[seq];
    const int pos0 = kv_len - q_len + t0;
    const int hi = pos0 + nt;
    const XsBlocks blocks = xs_blocks(pos0, hi, p.window, p.keep, BN);
    const int bs = (int)((int64_t)blocks.count * split / p.splits);           // this CTA's share, as indices of `blocks`
    const int be = (int)((int64_t)blocks.count * (split + 1) / p.splits);
    const int32_t* table = p.page_table + (int64_t)seq * p.P;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int G = p.G;
    const int rows_valid = nt * G;          // <= 16
    {
        constexpr int kLines = BN * D * 2 / 128, vLines = BN * DV * 2 / 128;      // 128-byte lines of one block of keys, of values
        const int lines = own_v ? kLines + vLines : kLines;
        for (int b = bs; b < min(be, bs + p.prefetch_blocks); ++b) {
            const int page = table[blocks.at(b)];
            if (page < 0) continue;
            const __nv_bfloat16* base = p.pool + (int64_t)page * p.Hkv * BN * (own_v ? D + DV : D);
            const __nv_bfloat16* kbase = base + (int64_t)kvh * BN * D;
            const __nv_bfloat16* vbase = base + (int64_t)p.Hkv * BN * D + (int64_t)kvh * BN * DV;
            for (int i = threadIdx.x; i < lines; i += NTHREADS) {
                const __nv_bfloat16* at = i < kLines ? kbase + i * 64 : vbase + (i - kLines) * 64;
                asm volatile("prefetch.global.L2 [%0];" ::"l"(at));
            }
        }
    }
    // this CTA's page numbers in one coalesced read (in pieces of 64 blocks); the first piece before the wait: the
    // page table is part of the step's description
    auto load_pages = [&](int from) {
        __syncthreads();
        if (threadIdx.x < 64 && from + (int)threadIdx.x < be) pages_sm[threadIdx.x] = table[blocks.at(from + threadIdx.x)];
        __syncthreads();
    };
    int pages_from = bs;
    load_pages(pages_from);
    pdl_wait();

    for (int c = threadIdx.x; c < QROWS * CHUNKS; c += NTHREADS) {
        const int r = c / CHUNKS, ch = c % CHUNKS;
        const bool ok = r < rows_valid;
        const int ti = ok ? r / G : 0, g = ok ? r % G : 0;
        const __nv_bfloat16* src = p.q + ((int64_t)(tok_begin + t0 + ti) * p.Hq + kvh * G + g) * D + ch * 8;
        cp_async16(q_sm + r * LD + ch * 8, src, ok);
    }
    auto load_block = [&](int i, int stage) {
        const int page = pages_sm[i - pages_from];
        load_kv_block<D, DV>(p, page, kvh, page >= 0 ? hi - blocks.at(i) * BN : 0, own_v, k_sm + stage * BN * LD, v_sm + stage * BN * LV);
    };
#pragma unroll
    for (int s = 0; s < NST - 1; ++s) {
        if (bs + s < be) load_block(bs + s, s);
        cp_async_commit();
    }

    const int r1 = lane >> 2, r2 = r1 + 8;
    const int pos1 = r1 < rows_valid ? pos0 + r1 / G : -1;
    const int pos2 = r2 < rows_valid ? pos0 + r2 / G : -1;
    const int lo1 = xs_first_visible(pos1, p.window), lo2 = xs_first_visible(pos2, p.window);     // found once: may cost a division
    float o[DTILES][4];
#pragma unroll
    for (int i = 0; i < DTILES; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m1 = -INFINITY, m2 = -INFINITY, l1 = 0.0f, l2 = 0.0f;
    unsigned qf[KSTEPS][4];
    bool q_loaded = false;

    for (int i_blk = bs, it = 0; i_blk < be; ++i_blk, ++it) {
        const int stage = it % NST, b = blocks.at(i_blk);
        cp_async_wait<NST - 2>();
        __syncthreads();
        const int nxt = i_blk + NST - 1;
        if (nxt < be) {
            if (nxt - pages_from >= 64) {          // the page numbers held do not reach that far: refill (rare: > 4,096 keys a split)
                cp_async_wait<0>();
                pages_from = i_blk;
                load_pages(pages_from);
            }
            load_block(nxt, (it + NST - 1) % NST);
        }
        cp_async_commit();
        if (!q_loaded) {
#pragma unroll
            for (int kk = 0; kk < KSTEPS; ++kk)
                ldmatrix_x4(qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], q_sm + (lane & 15) * LD + kk * 16 + (lane >> 4) * 8);
            q_loaded = true;
        }
        const __nv_bfloat16* ks = k_sm + stage * BN * LD + warp * 16 * LD;     // this warp's 16 keys of the block
        const __nv_bfloat16* vs = v_sm + stage * BN * LV + warp * 16 * LV;
        float s[2][4];
        s[0][0] = s[0][1] = s[0][2] = s[0][3] = s[1][0] = s[1][1] = s[1][2] = s[1][3] = 0.0f;
#pragma unroll
        for (int kk = 0; kk < KSTEPS; ++kk) {
            unsigned b0, b1, b2, b3;
            ldmatrix_x4(b0, b1, b2, b3, ks + ((lane >> 4) * 8 + (lane & 7)) * LD + kk * 16 + ((lane >> 3) & 1) * 8);
            mma_bf16(s[0], qf[kk], b0, b1);
            mma_bf16(s[1], qf[kk], b2, b3);
        }
        const float to_log2 = p.cap_out > 0.0f ? 1.0f : p.scale_log2;
        if (p.cap_out > 0.0f) xs_cap_scores<8>(&s[0][0], p.cap_in, p.cap_out);
        const int key0 = b * BN + warp * 16 + (lane & 3) * 2;
        float mx1 = -INFINITY, mx2 = -INFINITY;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int key = key0 + i * 8 + e;
                const bool v1 = key <= pos1 && (key >= lo1 || key < p.keep);
                const bool v2 = key <= pos2 && (key >= lo2 || key < p.keep);
                s[i][e] = v1 ? s[i][e] * to_log2 : -INFINITY;
                s[i][2 + e] = v2 ? s[i][2 + e] * to_log2 : -INFINITY;
                mx1 = fmaxf(mx1, s[i][e]);
                mx2 = fmaxf(mx2, s[i][2 + e]);
            }
        }
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        mx2 = fmaxf(mx2, __shfl_xor_sync(0xffffffffu, mx2, 1));
        mx2 = fmaxf(mx2, __shfl_xor_sync(0xffffffffu, mx2, 2));
        const float mn1 = fmaxf(m1, mx1), mn2 = fmaxf(m2, mx2);
        const float base1 = mn1 == -INFINITY ? 0.0f : mn1, base2 = mn2 == -INFINITY ? 0.0f : mn2;
        const float c1 = fast_exp2(m1 - base1), c2 = fast_exp2(m2 - base2);
        m1 = mn1;
        m2 = mn2;
        l1 *= c1;
        l2 *= c2;
#pragma unroll
        for (int i = 0; i < DTILES; ++i) {
            o[i][0] *= c1;
            o[i][1] *= c1;
            o[i][2] *= c2;
            o[i][3] *= c2;
        }
        unsigned pf[4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const float p0 = fast_exp2(s[i][0] - base1), p1 = fast_exp2(s[i][1] - base1);
            const float p2 = fast_exp2(s[i][2] - base2), p3 = fast_exp2(s[i][3] - base2);
            l1 += p0 + p1;
            l2 += p2 + p3;
            pf[i * 2 + 0] = pack_bf16(p0, p1);
            pf[i * 2 + 1] = pack_bf16(p2, p3);
        }
#pragma unroll
        for (int dp = 0; dp < DV / 16; ++dp) {
            unsigned b0, b1, b2, b3;
            ldmatrix_x4_trans(b0, b1, b2, b3, vs + (((lane >> 3) & 1) * 8 + (lane & 7)) * LV + dp * 16 + (lane >> 4) * 8);
            mma_bf16(o[2 * dp], pf, b0, b1);
            mma_bf16(o[2 * dp + 1], pf, b2, b3);
        }
    }
    cp_async_wait<0>();
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    l2 += __shfl_xor_sync(0xffffffffu, l2, 1);
    l2 += __shfl_xor_sync(0xffffffffu, l2, 2);

    // ---- merge the four warps: their outputs go through the (now idle) key stages
    __syncthreads();
    float* sm_o = reinterpret_cast<float*>(k_sm);          // [4][16][DV]
    if ((lane & 3) == 0) {
        sm_m[warp][r1] = m1;
        sm_l[warp][r1] = l1;
        sm_m[warp][r2] = m2;
        sm_l[warp][r2] = l2;
    }
#pragma unroll
    for (int i = 0; i < DTILES; ++i) {
        float* d1 = sm_o + ((warp * QROWS + r1) * DV) + i * 8 + (lane & 3) * 2;
        float* d2 = sm_o + ((warp * QROWS + r2) * DV) + i * 8 + (lane & 3) * 2;
        d1[0] = o[i][0];
        d1[1] = o[i][1];
        d2[0] = o[i][2];
        d2[1] = o[i][3];
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < rows_valid * DV; idx += NTHREADS) {
        const int r = idx / DV, d = idx % DV;
        float m = fmaxf(fmaxf(sm_m[0][r], sm_m[1][r]), fmaxf(sm_m[2][r], sm_m[3][r]));
        float l = 0.0f, acc = 0.0f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float f = sm_m[w][r] == -INFINITY ? 0.0f : fast_exp2(sm_m[w][r] - m);
            l += sm_l[w][r] * f;
            acc += sm_o[(w * QROWS + r) * DV + d] * f;
        }
        const int t = tok_begin + t0 + r / G, h = kvh * G + r % G;
        const int64_t row = (int64_t)t * p.Hq + h;
        if (p.splits == 1) {
            float f = inv_denominator(l, m, p.plus_one);
            if (p.gate != nullptr) f *= gate_of(p, t, p.gate_channels ? h * DV + d : h);
            p.out[(int64_t)t * p.ld_out + h * DV + d] = __float2bfloat16_rn(acc * f);
        } else {
            p.part_o[(row * p.splits + split) * DV + d] = acc;
            if (d == 0) {
                p.part_ml[(row * p.splits + split) * 2 + 0] = m;
                p.part_ml[(row * p.splits + split) * 2 + 1] = l;
            }
        }
    }
    if (p.splits == 1 || p.counters == nullptr) return;
    // ---- key splits without a kernel of their own to merge them: the CTA of a (sequence, kv head) that stores its part
    // last merges all of them (the same sums in the same order as attention_combine_kernel). Nobody waits for anybody.
    __shared__ bool is_last;
    __threadfence();
    __syncthreads();
    unsigned int* counter = p.counters + (int64_t)seq * p.Hkv + kvh;
    if (threadIdx.x == 0) is_last = atomicAdd(counter, 1u) == (unsigned)p.splits - 1;
    __syncthreads();
    if (!is_last) return;
    __threadfence();
    float* w_sm = reinterpret_cast<float*>(k_sm);            // [rows][64] weights, then [rows] 1 / sum (times a head's gate)
    float* f_sm = w_sm + QROWS * 64;
    for (int r = warp; r < rows_valid; r += NTHREADS / 32) {           // a warp a row; lane s holds splits s and s + 32
        const int t = tok_begin + t0 + r / G, h = kvh * G + r % G;
        const float* ml = p.part_ml + ((int64_t)t * p.Hq + h) * p.splits * 2;
        const float ms0 = lane < p.splits ? __ldcg(ml + 2 * lane) : -INFINITY;
        const float ms1 = lane + 32 < p.splits ? __ldcg(ml + 2 * (lane + 32)) : -INFINITY;
        const float ls0 = lane < p.splits ? __ldcg(ml + 2 * lane + 1) : 0.0f;
        const float ls1 = lane + 32 < p.splits ? __ldcg(ml + 2 * (lane + 32) + 1) : 0.0f;
        const float m = warp_max(fmaxf(ms0, ms1));
        const float wgt0 = ms0 == -INFINITY ? 0.0f : fast_exp2(ms0 - m);
        const float wgt1 = ms1 == -INFINITY ? 0.0f : fast_exp2(ms1 - m);
        const float l = warp_sum(ls0 * wgt0 + ls1 * wgt1);
        float f = inv_denominator(l, m, p.plus_one);
        if (p.gate != nullptr && !p.gate_channels) f *= gate_of(p, t, h);
        w_sm[r * 64 + lane] = wgt0;
        w_sm[r * 64 + 32 + lane] = wgt1;
        if (lane == 0) f_sm[r] = f;
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < rows_valid * (DV / 2); idx += NTHREADS) {
        const int r = idx / (DV / 2), d = (idx % (DV / 2)) * 2;
        const int t = tok_begin + t0 + r / G, h = kvh * G + r % G;
        const int64_t row = (int64_t)t * p.Hq + h;
        const float* po = p.part_o + row * p.splits * DV + d;
        float a0 = 0.0f, a1 = 0.0f;
#pragma unroll 8
        for (int s = 0; s < p.splits; ++s) {
            const float w = w_sm[r * 64 + s];
            const float2 raw = __ldcg(reinterpret_cast<const float2*>(po + (int64_t)s * DV));
            const float2 v = w == 0.0f ? make_float2(0.0f, 0.0f) : raw;      // an empty part's slot may hold anything
            a0 = fmaf(w, v.x, a0);
            a1 = fmaf(w, v.y, a1);
        }
        float f0 = f_sm[r], f1 = f0;
        if (p.gate_channels) {
            f0 *= gate_of(p, t, h * DV + d);
            f1 *= gate_of(p, t, h * DV + d + 1);
        }
        *reinterpret_cast<__nv_bfloat162*>(p.out + (int64_t)t * p.ld_out + h * DV + d) = __floats2bfloat162_rn(a0 * f0, a1 * f1);
    }
    if (threadIdx.x == 0) *counter = 0;          // ready for the next call
}

template <int D, int DV, int NST>
int launch_stages(const AttnParams& p, int max_tiles, int n_seqs, cudaStream_t stream) {
    constexpr size_t most = (size_t)((BM + NST * BN) * (D + 8) + NST * BN * (DV + 8)) * sizeof(__nv_bfloat16);
    const size_t smem = D == DV && p.planes == 1 ? (size_t)(BM + NST * BN) * (D + 8) * sizeof(__nv_bfloat16) : most;
    static bool opted = false;
    if (most > 48 * 1024 && !opted) {
        cudaFuncSetAttribute(attention_mma_kernel<D, DV, NST>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most);
        opted = true;
    }
    const dim3 grid(max_tiles, n_seqs, p.Hkv * p.splits);
    xs_launch(attention_mma_kernel<D, DV, NST>, grid, dim3(NTHREADS), smem, stream, p);
    return 0;
}

// Shared memory of the decode kernel: queries, stages of keys and (planes 2) values. The merge of the four warps takes
// [4][16][DV] floats of it, the merge of the key splits [16][65].
template <int D, int DV, int NST>
constexpr size_t decode_smem(int planes) {
    return (size_t)((16 + NST * BN) * (D + 8) + (D == DV && planes == 1 ? 0 : NST * BN * (DV + 8))) * sizeof(__nv_bfloat16);
}

template <int D, int DV, int NST>
int launch_decode(const AttnParams& p, int n_seqs, cudaStream_t stream) {
    constexpr size_t most = decode_smem<D, DV, NST>(2);
    const size_t smem = decode_smem<D, DV, NST>(p.planes);
    static bool opted = false;
    if (most > 48 * 1024 && !opted) {
        cudaFuncSetAttribute(attention_decode_mma_kernel<D, DV, NST>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most);
        opted = true;
    }
    const dim3 grid(1, n_seqs, p.Hkv * p.splits);
    xs_launch(attention_decode_mma_kernel<D, DV, NST>, grid, dim3(NTHREADS), smem, stream, p);
    return 0;
}

template <int D, int DV, int NST>
int decode_ctas_per_sm() {
    static int cached[16] = {};                  // per device: the answer does not change
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 16 && cached[dev] > 0) return cached[dev];
    constexpr size_t smem = decode_smem<D, DV, NST>(2);
    if (smem > 48 * 1024)
        cudaFuncSetAttribute(attention_decode_mma_kernel<D, DV, NST>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    int n = 0;
    if (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&n, attention_decode_mma_kernel<D, DV, NST>, NTHREADS, smem) != cudaSuccess)
        n = 0;
    if (dev >= 0 && dev < 16) cached[dev] = n;
    return n;
}

// Stages of the decode kernel for `tiles` (sequences x kv heads) CTAs before any key split. Three stages keep more
// of a CTA's keys in flight and win while the CTAs of one round fit the device (measured on B200, 8 sequences of
// 2,048 keys: 13.5 against 14.6 us). When even one CTA a tile is more than the three-stage kernel places at one
// time, two stages let five CTAs share an SM instead of three (64 sequences of 2,048 keys: 52.9 against 62.7 us).
template <int D, int DV>
int decode_stages_for(int64_t tiles) {
    if (g_attn_decode_stages <= 3) return g_attn_decode_stages < 3 ? 2 : 3;      // asked for by the caller
    return tiles > (int64_t)sm_count() * decode_ctas_per_sm<D, DV, 3>() ? 2 : 3;
}

template <int D, int DV>
int launch(const AttnParams& p, int max_tiles, int n_seqs, cudaStream_t stream) {
    if (p.decode_rows && decode_stages_for<D, DV>((int64_t)n_seqs * p.Hkv) >= 3) return launch_decode<D, DV, 3>(p, n_seqs, stream);
    if (p.decode_rows) return launch_decode<D, DV, 2>(p, n_seqs, stream);
    if constexpr (D == DV) {                 // (unequal sizes: one instance)
        if constexpr (D <= 64)
            if (max_tiles == 1 && g_attn_decode_stages >= 4) return launch_stages<D, DV, 4>(p, max_tiles, n_seqs, stream);
        if (max_tiles == 1 && g_attn_decode_stages >= 3) return launch_stages<D, DV, 3>(p, max_tiles, n_seqs, stream);
    }
    return launch_stages<D, DV, 2>(p, max_tiles, n_seqs, stream);
}

template <int D, int DV>
int decode_slots(int64_t tiles) {
    return sm_count() * (decode_stages_for<D, DV>(tiles) >= 3 ? decode_ctas_per_sm<D, DV, 3>() : decode_ctas_per_sm<D, DV, 2>());
}

// Unequal head sizes (attention_pairs.cu).
bool pair_supported(int D, int DV);
int launch_pair(const AttnParams& p, int D, int DV, int max_tiles, int n_seqs, cudaStream_t stream);     // -1: no such pair
int pair_decode_slots(int D, int DV, int64_t tiles);

}  // namespace xs_attn
