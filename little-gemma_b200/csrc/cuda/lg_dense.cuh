// lg_dense.cuh -- kernels over dense (bf16 or f32) weight matrices: the small-M matmul of a decode / verify step, the wide
// matmul of the prompt pass on tcgen05, their 32-bit counterpart, row norms with the residual update, embedding gather and
// rotation tables.
//
// A matrix is row-major [rows][ldk], ldk a multiple of 64 with zero padding behind the k columns, so every kernel walks whole
// chunks and whatever (finite) value an activation buffer holds behind its valid columns is multiplied by zero.
#pragma once
#include <cuda_bf16.h>
#include "lg_device.cuh"

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ void to_elem(float v, float &o) { o = v; }
__device__ __forceinline__ void to_elem(float v, bf16 &o) { o = __float2bfloat16_rn(v); }
__device__ __forceinline__ float from_elem(float v) { return v; }
__device__ __forceinline__ float from_elem(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) { __nv_bfloat162 v = __floats2bfloat162_rn(a, b); return *(uint32_t *)&v; }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + __expf(-z)); }
// activations of enum lg_act: value * gate of a gated unit, and the square of ReLU
__device__ __forceinline__ float gated_unit(float gate, float up) { return fmaxf(gate, 0.0f) * up; }
__device__ __forceinline__ float relu2_unit(float up) { const float r = fmaxf(up, 0.0f); return r * r; }

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// ---------------------------------------------------------------------------------------------
// pieces of latent attention that ride along with a matmul or stand alone
// ---------------------------------------------------------------------------------------------
// One position's cached row: [ RMS-normed latent (kv_rank) | 0 | rotated key part (rot_dim) | 0 ], the two parts starting at
// multiples of 16 elements.
struct LgCacheRow {
    const float *src; int ld;        // projection rows: latent at kv_off, key part at rot_off
    int kv_off, rot_off;
    const float *norm_w; float eps;
    int kv_rank, rot_dim, rot_dims;
    const float2 *tab;               // [tok][rot_dims / 2] cos, sin
    void *cache; int ldc, rot_at;    // row p of the cache starts at p * ldc
    const int *pos;                  // position of token 0
};
// The rotated part of every head's query, into the (absorbed) query rows the attention kernels over the cache read.
struct LgRotQ {
    const void *q; int ldq, head_stride, rot_at_q;
    void *out; int ldc, rot_at;      // out[(tok * H + h) * ldc + rot_at ..]
    int H, rot_dim, rot_dims;
    const float2 *tab;
};
// by all threads of a block; `red` >= 32 floats
template <typename T>
__device__ __forceinline__ void cache_row(const LgCacheRow &a, int tok, float *red) {
    const float *s = a.src + (size_t)tok * a.ld;
    T *row = (T *)a.cache + (size_t)(*a.pos + tok) * a.ldc;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.kv_rank; i += blockDim.x) { const float v = s[a.kv_off + i]; ss += v * v; }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)a.kv_rank + a.eps);
    for (int i = threadIdx.x; i < a.kv_rank; i += blockDim.x) to_elem(s[a.kv_off + i] * inv * a.norm_w[i], row[i]);
    const int half = a.rot_dims >> 1;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float u = s[a.rot_off + 2 * i], v = s[a.rot_off + 2 * i + 1];
        const float2 cs = a.tab[(size_t)tok * half + i];
        to_elem(u * cs.x - v * cs.y, row[a.rot_at + 2 * i]);
        to_elem(v * cs.x + u * cs.y, row[a.rot_at + 2 * i + 1]);
    }
    for (int i = a.rot_dims + threadIdx.x; i < a.rot_dim; i += blockDim.x) to_elem(s[a.rot_off + i], row[a.rot_at + i]);
}
template <typename T>
__device__ __forceinline__ void rot_q_rows(const LgRotQ &a, int tok, int first, int stride) {
    const int half = a.rot_dims >> 1, rest = a.rot_dim - a.rot_dims, per = half + rest;
    for (int u = first; u < a.H * per; u += stride) {
        const int h = u / per, i = u % per;
        const T *src = (const T *)a.q + (size_t)tok * a.ldq + (size_t)h * a.head_stride + a.rot_at_q;
        T *dst = (T *)a.out + ((size_t)tok * a.H + h) * a.ldc + a.rot_at;
        if (i < half) {
            const float x = from_elem(src[2 * i]), y = from_elem(src[2 * i + 1]);
            const float2 cs = a.tab[(size_t)tok * half + i];
            to_elem(x * cs.x - y * cs.y, dst[2 * i]);
            to_elem(y * cs.x + x * cs.y, dst[2 * i + 1]);
        } else dst[a.rot_dims + i - half] = src[a.rot_dims + i - half];
    }
}

// the same inside the query rows themselves (q == out)
__device__ __forceinline__ void rot_q_in_place(const LgRotQ &a, int tok, int first, int stride) {
    const int half = a.rot_dims >> 1;
    for (int u = first; u < a.H * half; u += stride) {
        const int h = u / half, i = u % half;
        uint32_t *p = (uint32_t *)((bf16 *)a.out + (size_t)tok * a.ldq + (size_t)h * a.head_stride + a.rot_at_q) + i;
        const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *)p), cs = a.tab[(size_t)tok * half + i];
        *p = pack_bf16(x.x * cs.x - x.y * cs.y, x.y * cs.x + x.x * cs.y);
    }
}

// ---------------------------------------------------------------------------------------------
// small-M matmul: out[tok][row] = W x[tok] for M <= 8 rows at once, bf16 weights streamed once
// ---------------------------------------------------------------------------------------------
// A warp owns one 16-row tile and one of KS slices of k.  Lane (g, t) loads 16 contiguous bytes of rows g and g + 8 per chunk
// of 32 columns: its A fragments of two m16n8k16 products whose k order inside the chunk is permuted; the activations (the
// 8-column B operand) are read with the same permutation, 16 contiguous bytes of token g.  The weight loads of a warp's first
// batch are issued before the dependency wait.  A row's products are added in an order that depends on the matrix only,
// never on M.
// PAIR: two matrices of equal width stacked, the second (from tile split_tile on) with activations x2 and the ReLU-square
// epilogue into bf16 rows of its own -- the two input projections of a layer whose mixer and feed-forward run side by side.
enum { DN_STORE = 0, DN_GLU = 1, DN_HEAD = 2, DN_SIGMOID_GATE = 3, DN_PAIR = 4 };
enum { DN_JOB_NONE = 0, DN_JOB_CACHE_ROW = 1, DN_JOB_ROT_Q = 2 };
#define DN_GEMV_THREADS 256
#define DN_GEMV_U 8                 // chunks of a batch: 16 loads of 16 bytes per lane in flight

struct LgDnGemvArgs {
    const bf16 *w; int ldk, n_tiles, rows;      // n_tiles = 16-row tiles; rows: valid rows (head)
    const bf16 *x; int ldx;                     // activations, when no norm is fused
    const float *xf; int ldxf, kx; const float *rms_w; float eps;   // RMSX: x = rms_norm(xf) * rms_w, rounded to bf16
    int tiles_per_group, x_group, out_group;    // rows in groups of so many tiles (0: one group), each with its own activations, at
                                                // + group * x_group, and its own stretch of the output row, at + group * out_group
    int M, n_main;                              // CTAs [n_main, gridDim.x) do the job below, one token each
    float *out; int ldo;                        // f32 rows
    bf16 *outh; int ldoh;                       // bf16 rows (instead of, or beside, out)
    const float *gate; int ld_gate;             // SIGMOID_GATE: outh = acc * sigmoid(gate)
    float *amax_val; int *amax_idx;             // HEAD: [n_main][LG_MAXM] best logit and row of each CTA
    int job; LgCacheRow cr; LgRotQ rq;
    const bf16 *x2; int split_tile;             // PAIR
    float out_scale = 1.0f;                     // HEAD: logits = out_scale * W x
};

template <int EPI, int KS, bool RMSX>
__global__ void __launch_bounds__(DN_GEMV_THREADS, 2) lg_dn_gemv_kernel(LgDnGemvArgs a) {
    extern __shared__ __align__(16) unsigned char dn_smem[];
    __shared__ float red[8][16][9];
    __shared__ float s_red[32];
    constexpr int TPC = 8 / KS, U = DN_GEMV_U;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int sub = warp / KS, ks = warp % KS;
    pdl_launch();
    if (blockIdx.x >= (unsigned)a.n_main) {
        pdl_wait();
        const int tok = blockIdx.x - a.n_main;
        if (a.job == DN_JOB_CACHE_ROW) cache_row<bf16>(a.cr, tok, s_red);
        else if (a.job == DN_JOB_ROT_Q) rot_q_rows<bf16>(a.rq, tok, threadIdx.x, blockDim.x);
        return;
    }
    const int nchunk = a.ldk >> 5;
    const int lo = (int)((long long)nchunk * ks / KS), hi = (int)((long long)nchunk * (ks + 1) / KS);
    uint4 w0[U], w1[U];
    auto load_batch = [&](int tile, int c) {
        const bf16 *p = a.w + ((size_t)tile * 16 + g) * a.ldk + c * 32 + t * 8;
        const size_t r8 = (size_t)8 * a.ldk;
        #pragma unroll
        for (int u = 0; u < U; u++) {
            if (c + u < hi) { w0[u] = ldg_stream16((const uint4 *)(p + u * 32)); w1[u] = ldg_stream16((const uint4 *)(p + r8 + u * 32)); }
            else { w0[u] = make_uint4(0, 0, 0, 0); w1[u] = make_uint4(0, 0, 0, 0); }
        }
    };
    int tile0 = blockIdx.x * TPC;
    const bool any = tile0 + sub < a.n_tiles;
    if (any) load_batch(tile0 + sub, lo);
    pdl_wait();

    const bf16 *xs = nullptr;
    const int ldxs = a.ldk + 8;                  // + 8: rows of the staged activations start in different banks
    if (RMSX) {
        bf16 *st = (bf16 *)dn_smem;
        for (int tok = 0; tok < a.M; tok++) {
            const float *src = a.xf + (size_t)tok * a.ldxf;
            float ss = 0.0f;
            for (int i = threadIdx.x; i < a.kx; i += DN_GEMV_THREADS) ss += src[i] * src[i];
            const float inv = 1.0f / sqrtf(block_sum(ss, s_red) / (float)a.kx + a.eps);
            for (int i = threadIdx.x; i < a.ldk; i += DN_GEMV_THREADS)
                st[tok * ldxs + i] = __float2bfloat16_rn(i < a.kx ? src[i] * inv * a.rms_w[i] : 0.0f);
        }
        __syncthreads();
        xs = st;
    }
    float best = -INFINITY; int besti = 0x7fffffff;
    bool first = true;
    for (; tile0 < a.n_tiles; tile0 += a.n_main * TPC) {
        const int tile = tile0 + sub;
        float c[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        if (tile < a.n_tiles) {
            const bf16 *xp = RMSX ? xs + g * ldxs : a.x + (size_t)g * a.ldx + (a.tiles_per_group ? (size_t)(tile / a.tiles_per_group) * a.x_group : 0);
            if (EPI == DN_PAIR && tile >= a.split_tile) xp = a.x2 + (size_t)g * a.ldx;
            for (int c0 = lo; c0 < hi; c0 += U) {
                if (!first) load_batch(tile, c0);
                first = false;
                uint4 b[U];
                #pragma unroll
                for (int u = 0; u < U; u++) {
                    b[u] = make_uint4(0, 0, 0, 0);
                    if (g < a.M && c0 + u < hi) b[u] = *(const uint4 *)(xp + (c0 + u) * 32 + t * 8);
                }
                #pragma unroll
                for (int u = 0; u < U; u++) {
                    mma_bf16(c, w0[u].x, w1[u].x, w0[u].y, w1[u].y, b[u].x, b[u].y);
                    mma_bf16(c, w0[u].z, w1[u].z, w0[u].w, w1[u].w, b[u].z, b[u].w);
                }
            }
        }
        __syncthreads();                         // the previous tile's sums have been read
        red[warp][g][2 * t] = c[0]; red[warp][g][2 * t + 1] = c[1];
        red[warp][g + 8][2 * t] = c[2]; red[warp][g + 8][2 * t + 1] = c[3];
        __syncthreads();
        #pragma unroll
        for (int o = threadIdx.x; o < TPC * 128; o += DN_GEMV_THREADS) {
            const int r = o & 15, tok = (o >> 4) & 7, tl = o >> 7, tt = tile0 + tl;
            if (tok >= a.M || tt >= a.n_tiles) continue;
            float v = 0.0f, v8 = 0.0f;
            #pragma unroll
            for (int k = 0; k < KS; k++) {
                v += red[tl * KS + k][r][tok];
                if (EPI == DN_GLU) v8 += red[tl * KS + k][(r + 8) & 15][tok];
            }
            if (EPI == DN_GLU) {
                if (r < 8) a.outh[(size_t)tok * a.ldoh + tt * 8 + r] = __float2bfloat16_rn(gated_unit(v, v8));
            } else if (EPI == DN_PAIR) {
                if (tt < a.split_tile) a.out[(size_t)tok * a.ldo + tt * 16 + r] = v;
                else a.outh[(size_t)tok * a.ldoh + (tt - a.split_tile) * 16 + r] = __float2bfloat16_rn(relu2_unit(v));
            } else {
                int row = tt * 16 + r;
                if (a.tiles_per_group) row = (tt % a.tiles_per_group) * 16 + r + (tt / a.tiles_per_group) * a.out_group;
                if (EPI == DN_SIGMOID_GATE) a.outh[(size_t)tok * a.ldoh + row] = __float2bfloat16_rn(v * sigmoid_f(a.gate[(size_t)tok * a.ld_gate + row]));
                else if (EPI == DN_HEAD) {
                    if (row < a.rows) {
                        v *= a.out_scale;
                        if (a.out) a.out[(size_t)tok * a.ldo + row] = v;
                        if (v > best || (v == best && row < besti)) { best = v; besti = row; }
                    }
                } else {
                    if (a.out) a.out[(size_t)tok * a.ldo + row] = v;
                    if (a.outh) a.outh[(size_t)tok * a.ldoh + row] = __float2bfloat16_rn(v);
                }
            }
        }
    }
    if (EPI == DN_HEAD) {
        // thread = (row of the tile, token): merge the 16 rows of a token, then the two halves of the block
        #pragma unroll
        for (int o = 8; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o); const int oi = __shfl_xor_sync(0xffffffffu, besti, o);
            if (ov > best || (ov == best && oi < besti)) { best = ov; besti = oi; }
        }
        __shared__ float sv[16]; __shared__ int si[16];
        if ((threadIdx.x & 15) == 0) { sv[threadIdx.x >> 4] = best; si[threadIdx.x >> 4] = besti; }
        __syncthreads();
        if (threadIdx.x < a.M) {
            float v = sv[threadIdx.x]; int i = si[threadIdx.x];
            const float ov = sv[threadIdx.x + 8]; const int oi = si[threadIdx.x + 8];
            if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
            a.amax_val[(size_t)blockIdx.x * LG_MAXM + threadIdx.x] = v;
            a.amax_idx[(size_t)blockIdx.x * LG_MAXM + threadIdx.x] = i;
        }
    }
}

// ---------------------------------------------------------------------------------------------
// wide matmul on tcgen05: out[tok][row] = W x[tok], bf16 operands, f32 accumulation in tensor memory
// ---------------------------------------------------------------------------------------------
// One CTA owns 128 tokens (the TMEM lanes) x NT weight rows (TMEM columns) and walks k in blocks of 64:
//   warp 4 (one thread)  loads the activation and the weight tile of a block with tiled TMA copies (128-byte swizzle); the
//                        weight tiles of the first stages are requested before the dependency wait;
//   warp 5 (one thread)  issues four tcgen05.mma (M = 128, N = NT, K = 16) per block and commits the stage back;
//   warps 0-3            read the accumulator (lane = token) and store 32 columns at a time with 16-byte stores.
enum { DN_G_F32 = 0, DN_G_BF16 = 1, DN_G_GLU = 2, DN_G_RELU2 = 3 };
#define DN_GEMM_BM 128
#define DN_GEMM_BK 64
#define DN_GEMM_THREADS 192
template <int NT> __host__ __device__ constexpr int dn_gemm_stages() { return NT == 256 ? 4 : 3; }
template <int NT> __host__ __device__ constexpr size_t dn_gemm_smem() {
    return 1024 + (size_t)dn_gemm_stages<NT>() * (DN_GEMM_BM + NT) * 128 + 256;
}
struct LgDnGemmArgs {
    int nkb, n_tok, cols;            // blocks of k; valid tokens; stored columns (a multiple of 32)
    int w_early;                     // the second operand does not depend on earlier kernels
    void *out; int ldo;              // f32 / bf16 rows; GLU: bf16 rows of cols / 2
    int *err;
    float out_scale = 1.0f;          // F32: out = out_scale * W x
    int f32_from = 0x7fffffff; float *out2 = nullptr; int ldo2 = 0;      // BF16: columns from here on (a multiple of 32) go to f32 rows of their own
};

template <int NT, int EPI>
__global__ void __launch_bounds__(DN_GEMM_THREADS) lg_dn_gemm_kernel(const __grid_constant__ CUtensorMap tmx, const __grid_constant__ CUtensorMap tmw,
                                                                      LgDnGemmArgs a) {
    extern __shared__ unsigned char dn_smem[];
    constexpr int ST = dn_gemm_stages<NT>(), A_BYTES = DN_GEMM_BM * 128, B_BYTES = NT * 128;
    unsigned char *base = (unsigned char *)(((uintptr_t)dn_smem + 1023) & ~(uintptr_t)1023);
    unsigned char *sA = base, *sB = base + ST * A_BYTES;
    uint64_t *full = (uint64_t *)(sB + ST * B_BYTES), *empty = full + ST, *acc_full = empty + ST;
    uint32_t *tmem_slot = (uint32_t *)(acc_full + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row0 = blockIdx.x * NT, tok0 = blockIdx.y * DN_GEMM_BM, nkb = a.nkb;

    if (threadIdx.x == 0) {
        for (int i = 0; i < ST; i++) { mbar_init(full + i, 1); mbar_init(empty + i, 1); }
        mbar_init(acc_full, 1);
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(smem_u32(tmem_slot)), "r"(NT) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;
    pdl_launch();                        // only now: a dependant must not take tensor memory a CTA of this grid still waits for

    if (warp == 4) {
        if (lane == 0) {
            const int pre = min(ST, nkb);
            if (!a.w_early) pdl_wait();
            for (int kb = 0; kb < pre; kb++) {
                mbar_expect_tx(full + kb, A_BYTES + B_BYTES);
                tma_load_2d(sB + kb * B_BYTES, &tmw, kb * DN_GEMM_BK, row0, full + kb);
            }
            if (a.w_early) pdl_wait();
            for (int kb = 0; kb < pre; kb++) tma_load_2d(sA + kb * A_BYTES, &tmx, kb * DN_GEMM_BK, tok0, full + kb);
            bool ok = true;
            int issued = pre;
            for (int kb = pre; kb < nkb && ok; kb++) {
                const int s = kb % ST;
                if (!mbar_wait(empty + s, ((kb / ST) & 1) ^ 1)) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 4); ok = false; break; }
                mbar_expect_tx(full + s, A_BYTES + B_BYTES);
                tma_load_2d(sB + s * B_BYTES, &tmw, kb * DN_GEMM_BK, row0, full + s);
                tma_load_2d(sA + s * A_BYTES, &tmx, kb * DN_GEMM_BK, tok0, full + s);
                issued = kb + 1;
            }
            if (!ok)      // drain: the copies already issued must land before the CTA's shared memory is released
                for (int kb = max(0, issued - ST); kb < issued; kb++) mbar_wait(full + kb % ST, (kb / ST) & 1);
        }
    } else if (warp == 5) {
        if (lane == 0) {
            // f32 accumulator, bf16 x bf16, both operands K-major
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NT >> 3) << 17) | ((uint32_t)(DN_GEMM_BM >> 4) << 24);
            bool ok = true;
            uint32_t acc = 0;
            for (int kb = 0; kb < nkb && ok; kb++) {
                const int s = kb % ST;
                if (!mbar_wait(full + s, (kb / ST) & 1)) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 8); ok = false; break; }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint64_t ad = umma_desc_k128(smem_u32(sA + s * A_BYTES)), bd = umma_desc_k128(smem_u32(sB + s * B_BYTES));
                #pragma unroll
                for (int j = 0; j < DN_GEMM_BK / 16; j++) { umma_f16(tmem, ad + 2 * j, bd + 2 * j, idesc, acc); acc = 1u; }
                umma_commit(empty + s);
            }
            umma_commit(acc_full);
        }
    } else {
        pdl_wait();                                // the outputs' earlier readers have finished
        const bool ok = mbar_wait(acc_full, 0);
        if (!ok && lane == 0) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 128);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const int tok = tok0 + warp * 32 + lane;
        if (ok)
            for (int c0 = 0; c0 < NT; c0 += 32) {
                const int col = row0 + c0;
                if (col >= a.cols) break;           // uniform per CTA
                uint32_t v[32];
                __syncwarp();
                tmem_ld32(tmem + ((uint32_t)(warp * 32) << 16) + c0, v);
                if (tok >= a.n_tok) continue;
                if (EPI == DN_G_F32) {
                    float4 *o = (float4 *)((float *)a.out + (size_t)tok * a.ldo + col);
                    #pragma unroll
                    for (int j = 0; j < 8; j++) o[j] = make_float4(__uint_as_float(v[4 * j]) * a.out_scale, __uint_as_float(v[4 * j + 1]) * a.out_scale, __uint_as_float(v[4 * j + 2]) * a.out_scale, __uint_as_float(v[4 * j + 3]) * a.out_scale);
                } else if (EPI == DN_G_BF16 && col >= a.f32_from) {
                    float4 *o = (float4 *)(a.out2 + (size_t)tok * a.ldo2 + col - a.f32_from);
                    #pragma unroll
                    for (int j = 0; j < 8; j++) o[j] = make_float4(__uint_as_float(v[4 * j]), __uint_as_float(v[4 * j + 1]), __uint_as_float(v[4 * j + 2]), __uint_as_float(v[4 * j + 3]));
                } else if (EPI == DN_G_RELU2) {
                    uint4 *o = (uint4 *)((bf16 *)a.out + (size_t)tok * a.ldo + col);
                    #pragma unroll
                    for (int j = 0; j < 4; j++) {
                        uint32_t p[4];
                        #pragma unroll
                        for (int i = 0; i < 4; i++) p[i] = pack_bf16(relu2_unit(__uint_as_float(v[8 * j + 2 * i])), relu2_unit(__uint_as_float(v[8 * j + 2 * i + 1])));
                        o[j] = make_uint4(p[0], p[1], p[2], p[3]);
                    }
                } else if (EPI == DN_G_BF16) {
                    uint4 *o = (uint4 *)((bf16 *)a.out + (size_t)tok * a.ldo + col);
                    #pragma unroll
                    for (int j = 0; j < 4; j++) {
                        const uint32_t *w = v + 8 * j;
                        o[j] = make_uint4(pack_bf16(__uint_as_float(w[0]), __uint_as_float(w[1])), pack_bf16(__uint_as_float(w[2]), __uint_as_float(w[3])),
                                          pack_bf16(__uint_as_float(w[4]), __uint_as_float(w[5])), pack_bf16(__uint_as_float(w[6]), __uint_as_float(w[7])));
                    }
                } else {
                    // columns come in groups of 8 gate rows and the 8 matching up rows
                    uint4 *o = (uint4 *)((bf16 *)a.out + (size_t)tok * a.ldo + col / 2);
                    #pragma unroll
                    for (int j = 0; j < 2; j++) {
                        uint32_t p[4];
                        #pragma unroll
                        for (int i = 0; i < 4; i++)
                            p[i] = pack_bf16(gated_unit(__uint_as_float(v[16 * j + 2 * i]), __uint_as_float(v[16 * j + 8 + 2 * i])),
                                             gated_unit(__uint_as_float(v[16 * j + 2 * i + 1]), __uint_as_float(v[16 * j + 9 + 2 * i])));
                        o[j] = make_uint4(p[0], p[1], p[2], p[3]);
                    }
                }
            }
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    }
    __syncthreads();
    if (warp == 5) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem), "r"(NT) : "memory");
    }
}

// ---------------------------------------------------------------------------------------------
// 32-bit matmul: out[tok][row] = W x[tok], f32 multiply-add (tiles of 64 tokens x 64 rows)
// ---------------------------------------------------------------------------------------------
struct LgDnF32Args {
    const float *w; int ldk; int rows, k;
    const float *x; int ldx, n;
    float *out; int ldo;
    size_t w_group; int x_group, out_group;      // blockIdx.z selects a group of rows with its own activations
    float out_scale = 1.0f;
};
__global__ void __launch_bounds__(256) lg_dn_gemm_f32_kernel(LgDnF32Args a) {
    __shared__ float sx[16][68], sw[16][68];
    pdl_launch(); pdl_wait();
    const float *W = a.w + blockIdx.z * a.w_group, *X = a.x + (size_t)blockIdx.z * a.x_group;
    float *O = a.out + (size_t)blockIdx.z * a.out_group;
    const int r0 = blockIdx.x * 64, t0 = blockIdx.y * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int li = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.k; k0 += 16) {
        #pragma unroll
        for (int j = 0; j < 4; j++) {
            const int k = k0 + lk + j;
            sw[lk + j][li] = r0 + li < a.rows && k < a.k ? W[(size_t)(r0 + li) * a.ldk + k] : 0.0f;
            sx[lk + j][li] = t0 + li < a.n && k < a.k ? X[(size_t)(t0 + li) * a.ldx + k] : 0.0f;
        }
        __syncthreads();
        #pragma unroll
        for (int k = 0; k < 16; k++) {
            float xv[4], wv[4];
            #pragma unroll
            for (int j = 0; j < 4; j++) { xv[j] = sx[k][ty * 4 + j]; wv[j] = sw[k][tx * 4 + j]; }
            #pragma unroll
            for (int i = 0; i < 4; i++)
                #pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
    #pragma unroll
    for (int i = 0; i < 4; i++)
        #pragma unroll
        for (int j = 0; j < 4; j++) {
            const int tok = t0 + ty * 4 + i, row = r0 + tx * 4 + j;
            if (tok < a.n && row < a.rows) O[(size_t)tok * a.ldo + row] = acc[i][j] * a.out_scale;
        }
}
// the 32-bit path's epilogues as kernels of their own
__global__ void lg_dn_glu_rows(const float *gu, int ld, int n_ff, float *out, int ldo) {      // groups of 8 gate, 8 up columns
    pdl_launch(); pdl_wait();
    const float *s = gu + (size_t)blockIdx.y * ld;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n_ff; i += gridDim.x * blockDim.x)
        out[(size_t)blockIdx.y * ldo + i] = gated_unit(s[(i >> 3) * 16 + (i & 7)], s[(i >> 3) * 16 + 8 + (i & 7)]);
}
__global__ void lg_dn_relu2_rows(const float *u, int ld, int n_ff, float *out, int ldo) {
    pdl_launch(); pdl_wait();
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n_ff; i += gridDim.x * blockDim.x)
        out[(size_t)blockIdx.y * ldo + i] = relu2_unit(u[(size_t)blockIdx.y * ld + i]);
}
__global__ void lg_dn_gate_rows(float *x, int ldx, const float *gate, int ldg, int n) {
    pdl_launch(); pdl_wait();
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x)
        x[(size_t)blockIdx.y * ldx + i] *= 1.0f / (1.0f + expf(-gate[(size_t)blockIdx.y * ldg + i]));
}
// argmax candidates of logits rows, the layout lg_argmax_final merges: [gridDim.x][LG_MAXM]
__global__ void lg_dn_argmax_rows(const float *logits, int ld, int n, float *val, int *idx) {
    pdl_launch(); pdl_wait();
    const float *s = logits + (size_t)blockIdx.y * ld;
    float bv = -INFINITY; int bi = 0x7fffffff;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x)
        if (s[i] > bv) { bv = s[i]; bi = i; }
    __shared__ float sv[8]; __shared__ int si[8];
    #pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o); const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
    if ((threadIdx.x & 31) == 0) { sv[threadIdx.x >> 5] = bv; si[threadIdx.x >> 5] = bi; }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < (int)(blockDim.x >> 5); w++) if (sv[w] > bv || (sv[w] == bv && si[w] < bi)) { bv = sv[w]; bi = si[w]; }
        val[(size_t)blockIdx.x * LG_MAXM + blockIdx.y] = bv; idx[(size_t)blockIdx.x * LG_MAXM + blockIdx.y] = bi;
    }
}

// ---------------------------------------------------------------------------------------------
// residual update + next norm, one CTA per token row
// ---------------------------------------------------------------------------------------------
// x += mult * norm(add) * add_w (add may be null), then y = norm(x) * norm_w.  The norm divides by the root of the mean square
// plus eps, after taking the mean off when `center` is set.  Every value of a row stays in registers between the passes.
// PAR (layers whose branches run side by side): x += add [+ bias] as they are, and two outputs with weights of their own.
struct LgRowNormArgs {
    float *x; int ldx, n;
    const float *add; int ld_add; const float *add_w; float mult;
    const float *norm_w; float eps; int center;
    void *y; int ldy;                // rows of T (norm_w null: not written)
    float *yf; int ldyf;             // optional f32 copy
    const float *bias;               // PAR: a vector added to the row, or null
    const float *norm_w2; void *y2;  // PAR: second output (null: none), leading dimension ldy
};
// V consecutive elements as one load / store
template <int V> struct alignas(V * 4) LgVec { float f[V]; };
template <int V> __device__ __forceinline__ LgVec<V> vec_load(const float *p) {
    LgVec<V> r;
    if (V == 4) *(float4 *)r.f = *(const float4 *)p; else r.f[0] = *p;
    return r;
}
template <int V> __device__ __forceinline__ void vec_store(float *p, const float *f) { if (V == 4) *(float4 *)p = *(const float4 *)f; else *p = *f; }
template <int V> __device__ __forceinline__ void vec_store(bf16 *p, const float *f) {
    if (V == 4) *(uint2 *)p = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[V - 1])); else *p = __float2bfloat16_rn(f[0]);
}
// item i of a thread: elements (tid + i * blockDim) * V ..
template <typename T, int IPT, int V, bool PAR = false>
__global__ void __launch_bounds__(1024) lg_row_norm_kernel(LgRowNormArgs a) {
    __shared__ float red[4][32];
    pdl_launch();
    LgVec<V> w1[IPT], w2[IPT], v[IPT], xv[IPT];
    const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, nw = (nt + 31) >> 5;
    auto zero = [](LgVec<V> &x) {
        #pragma unroll
        for (int j = 0; j < V; j++) x.f[j] = 0.0f;
    };
    auto fetch = [&](LgVec<V> (&d)[IPT], const float *p) {
        #pragma unroll
        for (int i = 0; i < IPT; i++) { const int c = (tid + i * nt) * V; if (p && c < a.n) d[i] = vec_load<V>(p + c); else zero(d[i]); }
    };
    fetch(w1, PAR ? a.norm_w2 : a.add ? a.add_w : nullptr);          // the weights do not depend on earlier kernels
    fetch(w2, a.norm_w);
    pdl_wait();
    float *x = a.x + (size_t)blockIdx.x * a.ldx;
    const float inv_n = 1.0f / (float)a.n;
    fetch(xv, x);
    fetch(v, a.add ? a.add + (size_t)blockIdx.x * a.ld_add : x);
    // sum over the row; each call has its own slots, so one barrier is enough
    auto row_sum = [&](float s, int slot) {
        s = warp_sum(s);
        if (lane == 0) red[slot][tid >> 5] = s;
        __syncthreads();
        return warp_sum(lane < nw ? red[slot][lane] : 0.0f);
    };
    // v <- (v - mean) / sqrt(mean of squared deviations + eps), in place
    auto normalise = [&](int slot) {
        if (a.center) {
            float s = 0.0f;
            #pragma unroll
            for (int i = 0; i < IPT; i++)
                #pragma unroll
                for (int j = 0; j < V; j++) s += v[i].f[j];
            const float mean = row_sum(s, slot) * inv_n;
            #pragma unroll
            for (int i = 0; i < IPT; i++)
                #pragma unroll
                for (int j = 0; j < V; j++) v[i].f[j] = (tid + i * nt) * V < a.n ? v[i].f[j] - mean : 0.0f;
        }
        float ss = 0.0f;
        #pragma unroll
        for (int i = 0; i < IPT; i++)
            #pragma unroll
            for (int j = 0; j < V; j++) ss += v[i].f[j] * v[i].f[j];
        const float inv = 1.0f / sqrtf(row_sum(ss, slot + 1) * inv_n + a.eps);
        #pragma unroll
        for (int i = 0; i < IPT; i++)
            #pragma unroll
            for (int j = 0; j < V; j++) v[i].f[j] *= inv;
    };
    if (PAR) {
        LgVec<V> b[IPT];
        fetch(b, a.bias);
        #pragma unroll
        for (int i = 0; i < IPT; i++) {
            const int c = (tid + i * nt) * V;
            #pragma unroll
            for (int j = 0; j < V; j++) xv[i].f[j] += (a.add ? v[i].f[j] : 0.0f) + b[i].f[j];
            if (c < a.n && (a.add || a.bias)) vec_store<V>(x + c, xv[i].f);
        }
    } else if (a.add) {
        normalise(0);
        #pragma unroll
        for (int i = 0; i < IPT; i++) {
            const int c = (tid + i * nt) * V;
            #pragma unroll
            for (int j = 0; j < V; j++) xv[i].f[j] += a.mult * (v[i].f[j] * w1[i].f[j]);
            if (c < a.n) vec_store<V>(x + c, xv[i].f);
        }
    }
    if (!a.norm_w) return;
    #pragma unroll
    for (int i = 0; i < IPT; i++) v[i] = xv[i];
    normalise(2);
    #pragma unroll
    for (int i = 0; i < IPT; i++) {
        const int c = (tid + i * nt) * V;
        if (c >= a.n) continue;
        alignas(V * 4) float y[V];
        #pragma unroll
        for (int j = 0; j < V; j++) y[j] = v[i].f[j] * w2[i].f[j];
        if (a.y) vec_store<V>((T *)a.y + (size_t)blockIdx.x * a.ldy + c, y);
        if (a.yf) vec_store<V>(a.yf + (size_t)blockIdx.x * a.ldyf + c, y);
        if (PAR && a.y2) {
            #pragma unroll
            for (int j = 0; j < V; j++) y[j] = v[i].f[j] * w1[i].f[j];
            vec_store<V>((T *)a.y2 + (size_t)blockIdx.x * a.ldy + c, y);
        }
    }
}

// ---------------------------------------------------------------------------------------------
// embedding rows, row gather, rotation tables
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void lg_dn_embed_rows(const T *w, int ldk, int n_rows, const int *toks, float *x, int n) {
    pdl_launch(); pdl_wait();
    const int id = min(max(toks[blockIdx.x], 0), n_rows - 1);
    for (int i = threadIdx.x; i < n; i += blockDim.x) x[(size_t)blockIdx.x * n + i] = from_elem(w[(size_t)id * ldk + i]);
}
// dst row i = src row idx[i]; rows of `bytes` bytes, a multiple of 16
__global__ void lg_dn_gather_rows(const void *src, const int *idx, void *dst, int bytes) {
    pdl_launch(); pdl_wait();
    const uint4 *s = (const uint4 *)((const char *)src + (size_t)idx[blockIdx.x] * bytes);
    uint4 *d = (uint4 *)((char *)dst + (size_t)blockIdx.x * bytes);
    for (int i = threadIdx.x; i < bytes / 16; i += blockDim.x) d[i] = s[i];
}
// tab[s][tok][i] = (cos, sin)((pos + tok) * base_s^(-2i / dims_s)) for every distinct rotation of the model (blockIdx.y = s).
// freq holds the powers; the angle is reduced in double so that its error does not grow with the position.
struct LgRotSpec { const double *freq; int half; float2 *tab; };
struct LgRotTables { LgRotSpec s[8]; const int *pos; int n_tok; };
__global__ void lg_dn_rot_tables(LgRotTables a) {
    pdl_launch(); pdl_wait();
    const LgRotSpec s = a.s[blockIdx.y];
    for (int u = blockIdx.x * blockDim.x + threadIdx.x; u < a.n_tok * s.half; u += gridDim.x * blockDim.x) {
        const int tok = u / s.half, i = u % s.half;
        const double turns = (double)(*a.pos + tok) * s.freq[i] * 0.15915494309189535;       // angle / 2 pi
        const float ang = (float)((turns - rint(turns)) * 6.283185307179586);
        s.tab[u] = make_float2(cosf(ang), sinf(ang));
    }
}
