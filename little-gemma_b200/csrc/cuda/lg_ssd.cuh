// lg_ssd.cuh -- a prompt block of a state-space layer in chunks of 128 tokens, as matrix products on tcgen05.
//
// With a_t the running sum of -exp(A_log) dt over a chunk, P[t][s] = (C_t . B_s) exp(a_t - a_s) dt_s for s <= t (plus D on the
// diagonal) and S the state before the chunk:
//     y_t = sum_s P[t][s] x_s + exp(a_t) S C_t,        S' = exp(a_last) S + sum_s exp(a_last - a_s) dt_s x_s B_s^T.
//  * lg_ssd_state_kernel: the sum of S' for every chunk and head;
//  * lg_ssd_scan_kernel:  S before every chunk, in f32 from chunk to chunk, left as bf16 high + low parts; the state behind the block;
//  * lg_ssd_out_kernel:   y.
// Step sizes, decays and sums are f32; what is f32 by nature and enters a product (P, the weighted x, S) enters as bf16 high + low
// parts; x, B and C are bf16 rows.  Tiles of 128 rows x 64 columns come by tiled TMA copies (128-byte swizzle); a tile whose rows
// are the contraction (tokens of x and B in S', state columns of S) is an MN-major operand.
#pragma once
#include "lg_seq.cuh"
#include "lg_latent.cuh"            // tensor-memory stores and products, high + low parts

#define LG_SSD_Q 128
#define LG_SSD_THREADS 128

// MN-major operand, 128-byte swizzle: rows of the contraction of 128 bytes (64 elements), 8-row groups 1024 bytes apart, blocks of 64
// columns `block` bytes apart
__device__ __forceinline__ uint64_t umma_desc_mn128(uint32_t saddr, uint32_t block) {
    return (uint64_t)((saddr & 0x3FFFFu) >> 4) | ((uint64_t)(block >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
#define LG_UMMA_A_MN (1u << 15)     // instruction descriptor: A / B stored MN-major
#define LG_UMMA_B_MN (1u << 16)
__device__ __forceinline__ void fence_async_shared() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

struct LgSsdArgs {
    const float *dt; int ld_dt;                  // raw step sizes [token][..]
    const float *dt_bias, *a_log, *d;
    int heads, groups, np, vdp, vs, n;           // vs: value columns per CTA (a multiple of 16, at most 128)
    float *ds, *decay;                           // [chunk][head][np][vdp] sums, [chunk][head] exp(a_last)
    bf16 *y; int ldy;                            // [token][heads vdp]
    int *err;
};
__host__ __device__ constexpr int lg_ssd_blocks(int cols) { return (cols + 63) / 64; }
__host__ __device__ constexpr size_t lg_ssd_state_smem(int np, int vs) {
    return 1024 + (size_t)(2 * ((np + 127) / 128) + 2 * lg_ssd_blocks(vs)) * LG_SSD_Q * 128 + 64;
}
__host__ __device__ constexpr size_t lg_ssd_out_smem(int np, int vs) {
    return 1024 + (size_t)(2 * lg_ssd_blocks(np) + lg_ssd_blocks(vs)) * LG_SSD_Q * 128 + (size_t)2 * lg_ssd_blocks(vs) * np * 128 + 64;
}
__host__ __device__ constexpr uint32_t lg_tmem_cols(int c) { return c <= 32 ? 32 : c <= 64 ? 64 : c <= 128 ? 128 : c <= 256 ? 256 : 512; }

// Step size and running log2 decay of the thread's token (thread = token of the chunk; tokens past the block: 0 and unchanged);
// returns the sum over the chunk.
__device__ __forceinline__ float chunk_decay(const LgSsdArgs &a, int h, int tok, float &dt, float &run, float *warp_tot) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    dt = tok < a.n ? softplus_f(a.dt[(size_t)tok * a.ld_dt + h] + a.dt_bias[h]) : 0.0f;
    run = -expf(a.a_log[h]) * dt * LG_LOG2E;
    #pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, run, o); if (lane >= o) run += v; }
    if (lane == 31) warp_tot[warp] = run;
    __syncthreads();
    const float t0 = warp_tot[0], t1 = warp_tot[1], t2 = warp_tot[2], t3 = warp_tot[3];
    run += warp == 0 ? 0.0f : warp == 1 ? t0 : warp == 2 ? t0 + t1 : t0 + t1 + t2;
    return t0 + t1 + t2 + t3;
}

// sums of B_s^T (w_s x_s) over a chunk: CTA (chunk, head, value slice); TMEM lane = state column
__global__ void __launch_bounds__(LG_SSD_THREADS) lg_ssd_state_kernel(const __grid_constant__ CUtensorMap tmu, LgSsdArgs a) {
    extern __shared__ __align__(16) unsigned char ssd_smem[];
    __shared__ float warp_tot[4];
    constexpr int BLK = LG_SSD_Q * 128;
    const int bm = (a.np + 127) / 128, xb = lg_ssd_blocks(a.vs);
    unsigned char *sB = (unsigned char *)(((uintptr_t)ssd_smem + 1023) & ~(uintptr_t)1023), *sX = sB + 2 * bm * BLK, *sL = sX + xb * BLK;
    uint64_t *full = (uint64_t *)(sL + xb * BLK), *done = full + 1;
    uint32_t *slot = (uint32_t *)(done + 1);
    const int tid = threadIdx.x, warp = tid >> 5, chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * a.vs, vs = min(a.vs, a.vdp - v0);
    const int g = h / (a.heads / a.groups), inner = a.heads * a.vdp, tok = chunk * LG_SSD_Q + tid;
    const uint32_t cols = lg_tmem_cols(bm * ((a.vs + 31) & ~31));
    if (tid == 0) { mbar_init(full, 1); mbar_init(done, 1); }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(smem_u32(slot)), "r"(cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *slot;
    pdl_launch();                        // only now: a dependant must not take tensor memory a CTA of this grid still waits for
    pdl_wait();
    const int nb = lg_ssd_blocks(a.np), nx = lg_ssd_blocks(vs);
    if (tid == 0) {
        mbar_expect_tx(full, (nb + nx) * BLK);
        for (int c = 0; c < nb; c++) tma_load_2d(sB + c * BLK, &tmu, inner + g * a.np + c * 64, chunk * LG_SSD_Q, full);
        for (int c = 0; c < nx; c++) tma_load_2d(sX + c * BLK, &tmu, h * a.vdp + v0 + c * 64, chunk * LG_SSD_Q, full);
    }
    float dt, run;
    const float last = chunk_decay(a, h, tok, dt, run, warp_tot);
    const float w = dt * exp2f(last - run);
    if (tid == 0 && blockIdx.z == 0) a.decay[(size_t)chunk * a.heads + h] = exp2f(last);
    bool ok = mbar_wait(full, 0);
    // row tid of x times its weight, high part in place
    if (ok)
        for (int c = 0; c < vs / 8; c++) {
            const uint32_t at = (uint32_t)(c >> 3) * BLK + tid * 128 + (((c & 7) ^ (tid & 7)) << 4);
            const uint4 u = *(const uint4 *)(sX + at);
            uint4 hi, lo;
            auto part = [&](uint32_t x, uint32_t &ph, uint32_t &pl) {
                const float2 f = __bfloat1622float2(*(const __nv_bfloat162 *)&x);
                if (tok < a.n) split_bf16(f.x * w, f.y * w, ph, pl); else ph = pl = 0;
            };
            part(u.x, hi.x, lo.x); part(u.y, hi.y, lo.y); part(u.z, hi.z, lo.z); part(u.w, hi.w, lo.w);
            *(uint4 *)(sX + at) = hi;
            *(uint4 *)(sL + at) = lo;
        }
    fence_async_shared();
    ok = __syncthreads_and(ok);
    const int ts = (a.vs + 31) & ~31;                // tensor-memory columns per tile of 128 state columns
    if (tid == 0 && ok) {
        const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(vs >> 3) << 17) | (8u << 24) | LG_UMMA_A_MN | LG_UMMA_B_MN;
        for (int m = 0; m < bm; m++) {
            const uint64_t bd = umma_desc_mn128(smem_u32(sB + 2 * m * BLK), BLK), xd = umma_desc_mn128(smem_u32(sX), BLK), ld = umma_desc_mn128(smem_u32(sL), BLK);
            for (int j = 0; j < LG_SSD_Q / 16; j++) {                // 16 tokens = 2048 bytes on
                umma_f16(tmem + m * ts, bd + j * 128, xd + j * 128, idesc, j ? 1u : 0u);
                umma_f16(tmem + m * ts, bd + j * 128, ld + j * 128, idesc, 1u);
            }
        }
        umma_commit(done);
    }
    if (ok) ok = mbar_wait(done, 0);
    ok = __syncthreads_and(ok);
    if (!ok && tid == 0) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 512);
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    if (ok)
        for (int m = 0; m < bm; m++) {
            const int nn = m * 128 + tid;
            float *o = a.ds + (((size_t)chunk * a.heads + h) * a.np + nn) * a.vdp + v0;
            for (int c = 0; c < vs; c += 32) {
                uint32_t v[32];
                __syncwarp();
                tmem_ld32(tmem + ((uint32_t)(warp * 32) << 16) + m * ts + c, v);
                if (nn >= a.np) continue;
                #pragma unroll
                for (int j = 0; j < 8; j++)
                    if (c + 4 * j < vs)
                        *(float4 *)(o + c + 4 * j) = make_float4(__uint_as_float(v[4 * j]), __uint_as_float(v[4 * j + 1]), __uint_as_float(v[4 * j + 2]), __uint_as_float(v[4 * j + 3]));
            }
        }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem), "r"(cols) : "memory");
    }
}

// S before every chunk: CTA = head x 32 state columns x 32 value rows; thread = 2 state columns x 2 value rows
struct LgSsdScanArgs {
    const float *ds, *decay; int heads, np, vdp, nst, chunks, fresh;
    float *state;                        // [head][vdp][nst]
    bf16 *hi, *lo;                       // [chunk][head][np][vdp]
};
#define LG_SSD_SCAN_THREADS 256
__global__ void __launch_bounds__(LG_SSD_SCAN_THREADS) lg_ssd_scan_kernel(LgSsdScanArgs a) {
    __shared__ float tile[32][33];
    pdl_launch(); pdl_wait();
    const int tid = threadIdx.x, h = blockIdx.x, n0 = blockIdx.y * 32, v0 = blockIdx.z * 32;
    float *st = a.state + ((size_t)h * a.vdp + v0) * a.nst + n0;
    if (!a.fresh)
        for (int i = tid; i < 1024; i += LG_SSD_SCAN_THREADS) tile[i >> 5][i & 31] = v0 + (i >> 5) < a.vdp ? st[(size_t)(i >> 5) * a.nst + (i & 31)] : 0.0f;
    __syncthreads();
    const int v = (tid & 15) * 2, nr = tid >> 4;
    float2 S[2];
    #pragma unroll
    for (int r = 0; r < 2; r++) S[r] = a.fresh ? make_float2(0.0f, 0.0f) : make_float2(tile[v][nr + 16 * r], tile[v + 1][nr + 16 * r]);
    const bool vok = v0 + v < a.vdp;
    const size_t per = (size_t)a.heads * a.np * a.vdp, at0 = ((size_t)h * a.np + n0 + nr) * a.vdp + v0 + v;
    #pragma unroll 4
    for (int c = 0; c < a.chunks; c++) {
        const float dec = a.decay[(size_t)c * a.heads + h];
        #pragma unroll
        for (int r = 0; r < 2; r++) {
            if (!vok || n0 + nr + 16 * r >= a.np) continue;
            const size_t at = at0 + c * per + (size_t)16 * r * a.vdp;
            const float2 d = *(const float2 *)(a.ds + at);
            uint32_t hi, lo;
            split_bf16(S[r].x, S[r].y, hi, lo);
            *(uint32_t *)(a.hi + at) = hi;
            *(uint32_t *)(a.lo + at) = lo;
            S[r].x = fmaf(dec, S[r].x, d.x);
            S[r].y = fmaf(dec, S[r].y, d.y);
        }
    }
    __syncthreads();
    #pragma unroll
    for (int r = 0; r < 2; r++) { tile[v][nr + 16 * r] = S[r].x; tile[v + 1][nr + 16 * r] = S[r].y; }
    __syncthreads();
    for (int i = tid; i < 1024; i += LG_SSD_SCAN_THREADS)
        if (v0 + (i >> 5) < a.vdp) st[(size_t)(i >> 5) * a.nst + (i & 31)] = n0 + (i & 31) < a.np ? tile[i >> 5][i & 31] : 0.0f;
}

// y of a chunk: CTA (chunk, head, value slice); TMEM lane = thread = token.  Columns 0..127: C B^T, then P over it (per 64 tokens 32
// columns of high parts, 32 of low parts); behind them P x and C S.
__global__ void __launch_bounds__(LG_SSD_THREADS) lg_ssd_out_kernel(const __grid_constant__ CUtensorMap tmu, const __grid_constant__ CUtensorMap tmh,
                                                                    const __grid_constant__ CUtensorMap tml, LgSsdArgs a) {
    extern __shared__ __align__(16) unsigned char ssd_smem[];
    __shared__ float warp_tot[4];
    __shared__ float2 col[LG_SSD_Q];                 // (running decay, step size) of every token
    constexpr int BLK = LG_SSD_Q * 128;
    const int nb = lg_ssd_blocks(a.np), xb = lg_ssd_blocks(a.vs), SBLK = a.np * 128;
    unsigned char *sC = (unsigned char *)(((uintptr_t)ssd_smem + 1023) & ~(uintptr_t)1023), *sB = sC + nb * BLK, *sX = sB + nb * BLK, *sH = sX + xb * BLK,
                  *sL = sH + xb * SBLK;
    uint64_t *full = (uint64_t *)(sL + xb * SBLK), *sfull = full + 1, *gdone = full + 2, *ydone = full + 3;
    uint32_t *slot = (uint32_t *)(full + 4);
    const int tid = threadIdx.x, warp = tid >> 5, chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * a.vs, vs = min(a.vs, a.vdp - v0);
    const int g = h / (a.heads / a.groups), inner = a.heads * a.vdp, tok = chunk * LG_SSD_Q + tid, ts = (a.vs + 31) & ~31;
    const uint32_t cols = lg_tmem_cols(LG_SSD_Q + 2 * ts);
    if (tid == 0) { mbar_init(full, 1); mbar_init(sfull, 1); mbar_init(gdone, 1); mbar_init(ydone, 1); }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(smem_u32(slot)), "r"(cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *slot, lanes = (uint32_t)(warp * 32) << 16, tY = tmem + LG_SSD_Q, tI = tY + ts;
    pdl_launch();
    pdl_wait();
    const int nx = lg_ssd_blocks(vs);
    if (tid == 0) {
        mbar_expect_tx(full, 2 * nb * BLK);
        for (int c = 0; c < nb; c++) {
            tma_load_2d(sC + c * BLK, &tmu, inner + (a.groups + g) * a.np + c * 64, chunk * LG_SSD_Q, full);
            tma_load_2d(sB + c * BLK, &tmu, inner + g * a.np + c * 64, chunk * LG_SSD_Q, full);
        }
        mbar_expect_tx(sfull, nx * BLK + 2 * nx * SBLK);
        for (int c = 0; c < nx; c++) {
            const int row = (chunk * a.heads + h) * a.np;
            tma_load_2d(sH + c * SBLK, &tmh, v0 + c * 64, row, sfull);
            tma_load_2d(sL + c * SBLK, &tml, v0 + c * 64, row, sfull);
            tma_load_2d(sX + c * BLK, &tmu, h * a.vdp + v0 + c * 64, chunk * LG_SSD_Q, sfull);
        }
    }
    float dt, run;
    chunk_decay(a, h, tok, dt, run, warp_tot);
    col[tid] = make_float2(run, dt);
    __syncthreads();
    const uint32_t fmt = (1u << 4) | (1u << 7) | (1u << 10) | (8u << 24);            // 128 rows, f32 accumulator, bf16 operands
    const uint32_t idY = fmt | ((uint32_t)(vs >> 3) << 17) | LG_UMMA_B_MN;
    bool ok = mbar_wait(full, 0) && mbar_wait(sfull, 0);
    ok = __syncthreads_and(ok);
    if (tid == 0 && ok) {
        const uint32_t idG = fmt | ((uint32_t)(LG_SSD_Q >> 3) << 17);
        const uint64_t cd = umma_desc_k128(smem_u32(sC)), bd = umma_desc_k128(smem_u32(sB));
        const uint64_t hd = umma_desc_mn128(smem_u32(sH), SBLK), ld = umma_desc_mn128(smem_u32(sL), SBLK);
        const int steps = a.np >> 4;
        for (int j = 0; j < steps; j++) umma_f16(tmem, cd + (j >> 2) * (BLK >> 4) + 2 * (j & 3), bd + (j >> 2) * (BLK >> 4) + 2 * (j & 3), idG, j ? 1u : 0u);
        umma_commit(gdone);
        for (int j = 0; j < steps; j++) {
            umma_f16(tI, cd + (j >> 2) * (BLK >> 4) + 2 * (j & 3), hd + j * 128, idY, j ? 1u : 0u);
            umma_f16(tI, cd + (j >> 2) * (BLK >> 4) + 2 * (j & 3), ld + j * 128, idY, 1u);
        }
    }
    if (ok) ok = mbar_wait(gdone, 0);
    ok = __syncthreads_and(ok);
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const float D = a.d[h];
    #pragma unroll 1
    for (int half = 0; half < 2 && ok; half++) {
        const uint32_t tG = tmem + lanes + half * 64;
        uint32_t s0[32], s1[32], hi[16], lo[16];
        __syncwarp();
        tmem_ld32(tG, s0);                             // all 64 columns, before the parts go over them
        tmem_ld32(tG + 32, s1);
        auto weigh = [&](const uint32_t (&s)[32], int first) {
            if (first > warp * 32 + 31) {              // all of it lies ahead of the warp's tokens
                #pragma unroll
                for (int j = 0; j < 16; j++) hi[j] = lo[j] = 0;
                return;
            }
            #pragma unroll
            for (int j = 0; j < 16; j++) {
                float p[2];
                #pragma unroll
                for (int i = 0; i < 2; i++) {
                    const int at = first + 2 * j + i;
                    const float2 cs = col[at];
                    p[i] = at <= tid ? __uint_as_float(s[2 * j + i]) * (ex2(run - cs.x) * cs.y) : 0.0f;
                    if (at == tid) p[i] += D;
                }
                split_bf16(p[0], p[1], hi[j], lo[j]);
            }
        };
        #pragma unroll
        for (int q = 0; q < 2; q++) {
            weigh(q ? s1 : s0, half * 64 + 32 * q);
            __syncwarp();
            tmem_st16(tG + 16 * q, hi);
            tmem_st16(tG + 32 + 16 * q, lo);
        }
    }
    tmem_wait_st();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    ok = __syncthreads_and(ok);
    if (tid == 0 && ok) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint64_t xd = umma_desc_mn128(smem_u32(sX), BLK);
        for (int half = 0; half < 2; half++)
            for (int j = 0; j < 4; j++) {
                umma_f16_ta(tY, tmem + half * 64 + 8 * j, xd + (half * 4 + j) * 128, idY, (half | j) ? 1u : 0u);
                umma_f16_ta(tY, tmem + half * 64 + 32 + 8 * j, xd + (half * 4 + j) * 128, idY, 1u);
            }
        umma_commit(ydone);
    }
    if (ok) ok = mbar_wait(ydone, 0);
    ok = __syncthreads_and(ok);
    if (!ok && tid == 0) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 1024);
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    if (ok) {
        const float er = ex2(run);
        bf16 *o = a.y + (size_t)tok * a.ldy + h * a.vdp + v0;
        for (int c = 0; c < vs; c += 32) {
            uint32_t y[32], z[32];
            __syncwarp();
            tmem_ld32(tY + lanes + c, y);
            tmem_ld32(tI + lanes + c, z);
            if (tok >= a.n) continue;
            auto val = [&](int j) { return fmaf(er, __uint_as_float(z[j]), __uint_as_float(y[j])); };
            #pragma unroll
            for (int j = 0; j < 4; j++)
                if (c + 8 * j < vs)
                    *(uint4 *)(o + c + 8 * j) = make_uint4(pack_bf16(val(8 * j), val(8 * j + 1)), pack_bf16(val(8 * j + 2), val(8 * j + 3)),
                                                           pack_bf16(val(8 * j + 4), val(8 * j + 5)), pack_bf16(val(8 * j + 6), val(8 * j + 7)));
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem), "r"(cols) : "memory");
    }
}
