// lg_ssd.cuh -- a prompt block of a state-space layer in chunks of 128 tokens, as matrix products on tcgen05.
//
// With a_t the running sum of -exp(A_log) dt over a chunk, P[t][s] = (C_t . B_s) exp(a_t - a_s) dt_s for s <= t (plus D on the
// diagonal) and S the state before the chunk:
//     y_t = sum_s P[t][s] x_s + exp(a_t) S C_t,        S' = exp(a_last) S + sum_s exp(a_last - a_s) dt_s x_s B_s^T.
//  * lg_ssd_state_kernel: S from chunk to chunk, as an accumulator in tensor memory; S before every chunk is left as bf16 high + low
//    parts, and the state behind the block;
//  * lg_ssd_out_kernel:   y.
// Step sizes, decays and sums are f32; what is f32 by nature and enters a product (P, the weighted x, S) enters as bf16 high + low
// parts; x, B and C are bf16 rows.  Tiles of 128 rows x 64 columns come by tiled TMA copies (128-byte swizzle); a tile whose rows
// are the contraction (tokens of x and B in S', state columns of S) is an MN-major operand.
#pragma once
#include "lg_seq.cuh"
#include "lg_latent.cuh"            // tensor-memory stores and products, high + low parts

#define LG_SSD_Q 128
#define LG_SSD_OUT_THREADS 448

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
    int heads, groups, np, vdp, vs, n;           // vs: value columns per CTA (a multiple of 16, at most 64)
    int splits, stages;                          // output kernel: parts that a group's heads are dealt into; stages of its tiles
    int nst, chunks, fresh;                      // columns of a stored state row; chunks of the block; a new sequence starts with it
    float *state;                                // [head][vdp][nst]
    bf16 *hi, *lo;                               // [chunk][head][np][vdp]
    bf16 *y; int ldy;                            // [token][heads vdp]
    int *err;
};
__host__ __device__ constexpr int lg_ssd_blocks(int cols) { return (cols + 63) / 64; }
#define LG_SSD_STATE_THREADS 576
#define LG_SSD_STAGES 3
__host__ __device__ constexpr size_t lg_ssd_state_smem(int vs) {
    return 1024 + (size_t)LG_SSD_STAGES * (2 + 2 * lg_ssd_blocks(vs)) * LG_SSD_Q * 128 + 256;
}
__host__ __device__ constexpr size_t lg_ssd_out_smem(int np, int stages) {
    return 1024 + (size_t)2 * lg_ssd_blocks(np) * LG_SSD_Q * 128 + (size_t)stages * (LG_SSD_Q + 2 * np) * 128 + 2 * LG_SSD_Q * 8 + 256;
}
__host__ __device__ constexpr uint32_t lg_tmem_cols(int c) { return c <= 32 ? 32 : c <= 64 ? 64 : c <= 128 ? 128 : c <= 256 ? 256 : 512; }

// Step size and running log2 decay of token `tok` (thread t of 128 in whole warps; tokens past the block: 0 and unchanged), from its raw
// step size; returns the sum over the chunk.  BAR: the named barrier of these threads.
template <int BAR>
__device__ __forceinline__ float chunk_decay(float raw, float bias, float A, int t, bool in, float &dt, float &run, float *warp_tot) {
    const int lane = t & 31, warp = t >> 5;
    dt = in ? softplus_f(raw + bias) : 0.0f;
    run = A * dt * LG_LOG2E;
    #pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, run, o); if (lane >= o) run += v; }
    if (lane == 31) warp_tot[warp] = run;
    asm volatile("bar.sync %0, 128;" :: "n"(BAR) : "memory");
    const float t0 = warp_tot[0], t1 = warp_tot[1], t2 = warp_tot[2], t3 = warp_tot[3];
    run += warp == 0 ? 0.0f : warp == 1 ? t0 : warp == 2 ? t0 + t1 : t0 + t1 + t2;
    return t0 + t1 + t2 + t3;
}

// States from chunk to chunk: CTA (head, value slice, 128 state columns); TMEM lane = state column, TMEM columns = value columns.
//   warps 0-3  state: what the accumulator holds before a chunk goes to memory as high + low parts and, times the chunk's decay, back into
//              the accumulator;
//   warps 4-15  in three groups, every third chunk, one token per thread: step sizes, running decay, the token's x times its weight as high (in place)
//              + low parts;
//   warp 16    (one thread) tiles of B and x;   warp 17  (one thread) the products of a chunk onto the accumulator.
__global__ void __launch_bounds__(LG_SSD_STATE_THREADS) lg_ssd_state_kernel(const __grid_constant__ CUtensorMap tmu, LgSsdArgs a) {
    extern __shared__ __align__(16) unsigned char ssd_smem[];
    __shared__ float warp_tot[3][2][4], s_dec[LG_SSD_STAGES];
    constexpr int BLK = LG_SSD_Q * 128, ST = LG_SSD_STAGES;
    const int xb = lg_ssd_blocks(a.vs);
    unsigned char *sB = (unsigned char *)(((uintptr_t)ssd_smem + 1023) & ~(uintptr_t)1023), *sX = sB + ST * 2 * BLK, *sL = sX + ST * xb * BLK;
    uint64_t *full = (uint64_t *)(sL + ST * xb * BLK), *xready = full + ST, *done = xready + ST, *sready = done + ST;
    uint32_t *slot = (uint32_t *)(sready + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.x, v0 = blockIdx.y * a.vs, vs = min(a.vs, a.vdp - v0), n0 = blockIdx.z * 128;
    const int g = h / (a.heads / a.groups), inner = a.heads * a.vdp;
    const uint32_t cols = lg_tmem_cols((a.vs + 31) & ~31);
    if (threadIdx.x == 0) {
        for (int i = 0; i < ST; i++) { mbar_init(full + i, 1); mbar_init(xready + i, 128); mbar_init(done + i, 1); }
        mbar_init(sready, 128);
    }
    if (warp == 17) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(smem_u32(slot)), "r"(cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *slot;
    pdl_launch();                        // only now: a dependant must not take tensor memory a CTA of this grid still waits for
    pdl_wait();
    const int nb = min(2, lg_ssd_blocks(a.np - n0)), nx = lg_ssd_blocks(vs);
    if (warp == 16) {
        if (lane == 0) {
            int c = 0;
            for (; c < a.chunks; c++) {
                const int s = c % ST;
                if (c >= ST && !mbar_wait(done + s, (c / ST - 1) & 1)) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 512); break; }
                mbar_expect_tx(full + s, (nb + nx) * BLK);
                for (int i = 0; i < nb; i++) tma_load_2d(sB + (2 * s + i) * BLK, &tmu, inner + g * a.np + n0 + i * 64, c * LG_SSD_Q, full + s);
                for (int i = 0; i < nx; i++) tma_load_2d(sX + (s * xb + i) * BLK, &tmu, h * a.vdp + v0 + i * 64, c * LG_SSD_Q, full + s);
            }
            if (c < a.chunks) for (int j = max(0, c - ST); j < c; j++) mbar_wait(full + j % ST, (j / ST) & 1);        // own copies in flight land before the CTA ends
        }
    } else if (warp == 17) {
        if (lane == 0) {
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(vs >> 3) << 17) | (8u << 24) | LG_UMMA_A_MN | LG_UMMA_B_MN;
            bool ok = true;
            for (int c = 0; c < a.chunks && ok; c++) {
                const int s = c % ST;
                ok = mbar_wait(full + s, (c / ST) & 1) && mbar_wait(xready + s, (c / ST) & 1) && mbar_wait(sready, c & 1);
                if (!ok) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 512); break; }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint64_t bd = umma_desc_mn128(smem_u32(sB + 2 * s * BLK), BLK), xd = umma_desc_mn128(smem_u32(sX + s * xb * BLK), BLK),
                               ld = umma_desc_mn128(smem_u32(sL + s * xb * BLK), BLK);
                #pragma unroll
                for (int j = 0; j < LG_SSD_Q / 16; j++) {                // 16 tokens = 2048 bytes on
                    umma_f16(tmem, bd + j * 128, xd + j * 128, idesc, 1u);
                    umma_f16(tmem, bd + j * 128, ld + j * 128, idesc, 1u);
                }
                umma_commit(done + s);
            }
        }
    } else if (warp >= 4) {
        const int t = threadIdx.x & 127, grp = (warp >> 2) - 1;
        const float bias = a.dt_bias[h], A = -expf(a.a_log[h]);
        float raw = grp * LG_SSD_Q + t < a.n ? a.dt[(size_t)(grp * LG_SSD_Q + t) * a.ld_dt + h] : 0.0f;
        bool ok = true;
        for (int c = grp; c < a.chunks; c += 3) {
            const int s = c % ST, tok = c * LG_SSD_Q + t, ahead = tok + 3 * LG_SSD_Q;
            const float next = ahead < a.n ? a.dt[(size_t)ahead * a.ld_dt + h] : 0.0f;
            float dt, run;
            float *tot = warp_tot[grp][(c / 3) & 1];
            const float last = grp == 0 ? chunk_decay<1>(raw, bias, A, t, tok < a.n, dt, run, tot) : grp == 1 ? chunk_decay<2>(raw, bias, A, t, tok < a.n, dt, run, tot)
                                                                                                     : chunk_decay<3>(raw, bias, A, t, tok < a.n, dt, run, tot);
            const float w = dt * exp2f(last - run);
            raw = next;
            ok = ok && mbar_wait(full + s, (c / ST) & 1);         // (requested once the products had used the stage)
            if (t == 0) s_dec[s] = exp2f(last);
            if (ok)
                for (int i = 0; i < vs / 8; i++) {
                    const uint32_t at = (uint32_t)(s * xb + (i >> 3)) * BLK + t * 128 + (((i & 7) ^ (t & 7)) << 4);
                    const uint4 u = *(const uint4 *)(sX + at);
                    uint4 hi, lo;
                    auto part = [&](uint32_t x, uint32_t &ph, uint32_t &pl) {
                        const float2 f = __bfloat1622float2(*(const __nv_bfloat162 *)&x);
                        if (tok < a.n) split_bf16(f.x * w, f.y * w, ph, pl); else ph = pl = 0;
                    };
                    part(u.x, hi.x, lo.x); part(u.y, hi.y, lo.y); part(u.z, hi.z, lo.z); part(u.w, hi.w, lo.w);
                    *(uint4 *)(sX + at) = hi;                     // in place
                    *(uint4 *)(sL + at) = lo;
                }
            fence_async_shared();
            mbar_arrive(xready + s);
        }
        if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 512);
    } else {
        const int nn = n0 + threadIdx.x;
        const uint32_t tS = tmem + ((uint32_t)(warp * 32) << 16);
        const bool mine = nn < a.np;
        float *st = a.state + ((size_t)h * a.vdp + v0) * a.nst + nn;
        for (int c = 0; c < vs; c += 32) {                              // where the block starts
            uint32_t v[32];
            #pragma unroll
            for (int j = 0; j < 32; j++) v[j] = !a.fresh && mine && c + j < vs ? __float_as_uint(st[(size_t)(c + j) * a.nst]) : 0u;
            __syncwarp();
            tmem_st32(tS + c, v);
        }
        tmem_wait_st();
        bool ok = true;
        for (int k = 0; k <= a.chunks; k++) {
            if (k) {
                ok = __all_sync(0xffffffffu, ok && mbar_wait(done + (k - 1) % ST, ((k - 1) / ST) & 1));
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            }
            if (k == a.chunks) break;
            ok = __all_sync(0xffffffffu, ok && mbar_wait(xready + k % ST, (k / ST) & 1));        // the chunk's decay is there
            const float dec = s_dec[k % ST];
            bf16 *hi = a.hi + (((size_t)k * a.heads + h) * a.np + nn) * a.vdp + v0, *lo = a.lo + (hi - a.hi);
            for (int c = 0; c < vs; c += 32) {
                uint32_t v[32], w[32];
                __syncwarp();
                tmem_ld32(tS + c, v);
                #pragma unroll
                for (int j = 0; j < 32; j++) w[j] = __float_as_uint(__uint_as_float(v[j]) * dec);
                tmem_st32(tS + c, w);
                if (c + 32 >= vs) {                    // the products may go on while the last columns are written out
                    tmem_wait_st();
                    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                    mbar_arrive(sready);
                }
                if (!mine) continue;
                #pragma unroll
                for (int j = 0; j < 4; j++)
                    if (c + 8 * j < vs) {
                        uint4 ph, pl;
                        auto part = [&](int i, uint32_t &x, uint32_t &y) { split_bf16(__uint_as_float(v[8 * j + i]), __uint_as_float(v[8 * j + i + 1]), x, y); };
                        part(0, ph.x, pl.x); part(2, ph.y, pl.y); part(4, ph.z, pl.z); part(6, ph.w, pl.w);
                        *(uint4 *)(hi + c + 8 * j) = ph;
                        *(uint4 *)(lo + c + 8 * j) = pl;
                    }
            }
        }
        if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 512);
        for (int c = 0; c < vs; c += 32) {
            uint32_t v[32];
            __syncwarp();
            tmem_ld32(tS + c, v);
            if (nn >= a.nst) continue;
            #pragma unroll
            for (int j = 0; j < 32; j++) if (c + j < vs) st[(size_t)(c + j) * a.nst] = mine ? __uint_as_float(v[j]) : 0.0f;
        }
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    }
    __syncthreads();
    if (warp == 17) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem), "r"(cols) : "memory");
    }
}

// y of a chunk: CTA (chunk, part of a group's heads, value slice); TMEM lane = token.  C B^T is multiplied once for all heads of the group; then
// head by head P over a buffer of its own (per 64 tokens 32 columns of high parts, 32 of low parts), P x and C S into one of two pairs of
// accumulators.
//   warps 0-7    P and, one head behind, the finished rows: warps 0-3 and 4-7 share a token's columns by halves;
//   warps 8-11   step sizes and running decay of the next head, one token per thread;
//   warp 12      (one thread) tiles: C and B once, x and S per head;   warp 13  (one thread) products.
__global__ void __launch_bounds__(LG_SSD_OUT_THREADS, 1) lg_ssd_out_kernel(const __grid_constant__ CUtensorMap tmu, const __grid_constant__ CUtensorMap tmh,
                                                                       const __grid_constant__ CUtensorMap tml, LgSsdArgs a) {
    extern __shared__ __align__(16) unsigned char ssd_smem[];
    __shared__ float warp_tot[2][4];
    constexpr int BLK = LG_SSD_Q * 128;
    const int nb = lg_ssd_blocks(a.np), ST = a.stages, SBLK = a.np * 128, SET = BLK + 2 * SBLK;
    unsigned char *sC = (unsigned char *)(((uintptr_t)ssd_smem + 1023) & ~(uintptr_t)1023), *sB = sC + nb * BLK, *sX = sB + nb * BLK;      // stage: [x | S high | S low]
    float2 (*col)[LG_SSD_Q] = (float2 (*)[LG_SSD_Q])(sX + ST * SET);              // [2]: (running decay, step size) of every token
    uint64_t *cbfull = (uint64_t *)(col + 2), *gdone = cbfull + 1, *pready = cbfull + 2, *full = cbfull + 3, *ydone = full + 2, *yfree = ydone + 2, *cready = yfree + 2,
             *cfree = cready + 2;
    uint32_t *slot = (uint32_t *)(cfree + 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, chunk = blockIdx.x, v0 = blockIdx.z * a.vs, vs = min(a.vs, a.vdp - v0);
    const int per = a.heads / a.groups, g = blockIdx.y / a.splits, part = blockIdx.y % a.splits, h0 = g * per + (int)((long long)per * part / a.splits),
              nh = g * per + (int)((long long)per * (part + 1) / a.splits) - h0, inner = a.heads * a.vdp;
    if (threadIdx.x == 0) {
        mbar_init(cbfull, 1); mbar_init(gdone, 1); mbar_init(pready, 256);
        for (int i = 0; i < 2; i++) { mbar_init(full + i, 1); mbar_init(ydone + i, 1); mbar_init(yfree + i, 256); mbar_init(cready + i, 128); mbar_init(cfree + i, 256); }
    }
    if (warp == 13) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(smem_u32(slot)), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *slot, tP = tmem + LG_SSD_Q, tA = tP + LG_SSD_Q;        // accumulator pair b: P x at tA + 128 b, C S 64 columns on
    pdl_launch();                        // only now: a dependant must not take tensor memory a CTA of this grid still waits for
    pdl_wait();
    if (warp == 12) {
        if (lane == 0) {
            mbar_expect_tx(cbfull, 2 * nb * BLK);
            for (int c = 0; c < nb; c++) {
                tma_load_2d(sC + c * BLK, &tmu, inner + (a.groups + g) * a.np + c * 64, chunk * LG_SSD_Q, cbfull);
                tma_load_2d(sB + c * BLK, &tmu, inner + g * a.np + c * 64, chunk * LG_SSD_Q, cbfull);
            }
            int i = 0;
            for (; i < nh; i++) {
                const int s = i % ST, used = i - ST, h = h0 + i, row = (chunk * a.heads + h) * a.np;
                if (used >= 0 && !mbar_wait(ydone + (used & 1), (used >> 1) & 1)) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 1024); break; }
                unsigned char *d = sX + s * SET;
                mbar_expect_tx(full + s, SET);
                tma_load_2d(d, &tmu, h * a.vdp + v0, chunk * LG_SSD_Q, full + s);
                tma_load_2d(d + BLK, &tmh, v0, row, full + s);
                tma_load_2d(d + BLK + SBLK, &tml, v0, row, full + s);
            }
            if (i < nh) { mbar_wait(cbfull, 0); for (int j = max(0, i - ST); j < i; j++) mbar_wait(full + j % ST, (j / ST) & 1); }      // own copies land before the CTA ends
        }
    } else if (warp == 13) {
        if (lane == 0) {
            const uint32_t fmt = (1u << 4) | (1u << 7) | (1u << 10) | (8u << 24);            // 128 rows, f32 accumulator, bf16 operands
            const uint32_t idG = fmt | ((uint32_t)(LG_SSD_Q >> 3) << 17), idY = fmt | ((uint32_t)(vs >> 3) << 17) | LG_UMMA_B_MN;
            const uint64_t cd = umma_desc_k128(smem_u32(sC)), bd = umma_desc_k128(smem_u32(sB));
            const int steps = a.np >> 4;
            bool ok = mbar_wait(cbfull, 0);
            if (ok) {
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                for (int j = 0; j < steps; j++) umma_f16(tmem, cd + (j >> 2) * (BLK >> 4) + 2 * (j & 3), bd + (j >> 2) * (BLK >> 4) + 2 * (j & 3), idG, j ? 1u : 0u);
                umma_commit(gdone);
            }
            for (int i = 0; i < nh && ok; i++) {
                const int s = i % ST, b = i & 1;
                ok = mbar_wait(full + s, (i / ST) & 1) && (i < 2 || mbar_wait(yfree + b, ((i >> 1) - 1) & 1));
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t xa = smem_u32(sX + s * SET), tY = tA + 128 * b, tI = tY + 64;
                const uint64_t xd = umma_desc_mn128(xa, BLK), hd = umma_desc_mn128(xa + BLK, SBLK), ld = umma_desc_mn128(xa + BLK + SBLK, SBLK);
                for (int j = 0; j < steps; j++) {
                    umma_f16(tI, cd + (j >> 2) * (BLK >> 4) + 2 * (j & 3), hd + j * 128, idY, j ? 1u : 0u);
                    umma_f16(tI, cd + (j >> 2) * (BLK >> 4) + 2 * (j & 3), ld + j * 128, idY, 1u);
                }
                ok = mbar_wait(pready, i & 1);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                #pragma unroll
                for (int j = 0; j < 8; j++) {
                    umma_f16_ta(tY, tP + (j >> 2) * 64 + 8 * (j & 3), xd + j * 128, idY, j ? 1u : 0u);
                    umma_f16_ta(tY, tP + (j >> 2) * 64 + 32 + 8 * (j & 3), xd + j * 128, idY, 1u);
                }
                umma_commit(ydone + b);
            }
            if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 1024);
        }
    } else if (warp >= 8) {
        const int t = threadIdx.x & 127, tok = chunk * LG_SSD_Q + t;
        bool ok = true;
        float raw = tok < a.n ? a.dt[(size_t)tok * a.ld_dt + h0] : 0.0f;
        for (int i = 0; i < nh; i++) {
            const int h = h0 + i;
            const float next = tok < a.n && i + 1 < nh ? a.dt[(size_t)tok * a.ld_dt + h + 1] : 0.0f;
            float dt, run;
            chunk_decay<1>(raw, a.dt_bias[h], -expf(a.a_log[h]), t, tok < a.n, dt, run, warp_tot[i & 1]);
            raw = next;
            ok = ok && (i < 2 || mbar_wait(cfree + (i & 1), ((i >> 1) - 1) & 1));
            col[i & 1][t] = make_float2(run, dt);
            mbar_arrive(cready + (i & 1));
        }
        if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 1024);
    } else {
        const int half = warp >> 2, t = threadIdx.x & 127, tok = chunk * LG_SSD_Q + t, first = half * 64, rows_end = (warp & 3) * 32 + 31;
        const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16, tG = tmem + lanes + first, tPw = tP + lanes + first;
        bool ok = __all_sync(0xffffffffu, mbar_wait(gdone, 0));
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        float run_before = 0.0f;
        for (int i = 0; i <= nh; i++) {
            float run = 0.0f;
            uint32_t hi[2][16], lo[2][16];
            if (i < nh) {
                ok = __all_sync(0xffffffffu, ok && mbar_wait(cready + (i & 1), (i >> 1) & 1));
                const float2 *cl = col[i & 1];
                run = cl[t].x;
                const float D = a.d[h0 + i];
                #pragma unroll
                for (int q = 0; q < 2; q++) {
                    if (first + 32 * q > rows_end) {           // all of it lies ahead of the warp's tokens
                        #pragma unroll
                        for (int j = 0; j < 16; j++) hi[q][j] = lo[q][j] = 0;
                        continue;
                    }
                    uint32_t sc[32];
                    __syncwarp();
                    tmem_ld32(tG + 32 * q, sc);
                    #pragma unroll
                    for (int j = 0; j < 16; j++) {
                        float p[2];
                        #pragma unroll
                        for (int x = 0; x < 2; x++) {
                            const int at = first + 32 * q + 2 * j + x;
                            const float2 cs = cl[at];
                            p[x] = at <= t ? __uint_as_float(sc[2 * j + x]) * (ex2(run - cs.x) * cs.y) : 0.0f;
                            if (at == t) p[x] += D;
                        }
                        split_bf16(p[0], p[1], hi[q][j], lo[q][j]);
                    }
                }
                mbar_arrive(cfree + (i & 1));
            }
            if (i) {
                ok = __all_sync(0xffffffffu, ok && mbar_wait(ydone + ((i - 1) & 1), ((i - 1) >> 1) & 1));          // the products of the head before are done
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            }
            if (i < nh) {
                __syncwarp();
                #pragma unroll
                for (int q = 0; q < 2; q++) { tmem_st16(tPw + 16 * q, hi[q]); tmem_st16(tPw + 32 + 16 * q, lo[q]); }
                tmem_wait_st();
                asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                mbar_arrive(pready);
            }
            if (i) {
                const uint32_t tY = tA + lanes + 128 * ((i - 1) & 1), tI = tY + 64;
                const float er = ex2(run_before);
                const int c = half * 32;
                if (c < vs) {
                    uint32_t y[32], z[32];
                    __syncwarp();
                    tmem_ld32(tY + c, y);
                    tmem_ld32(tI + c, z);
                    if (tok < a.n && ok) {
                        bf16 *o = a.y + (size_t)tok * a.ldy + (h0 + i - 1) * a.vdp + v0 + c;
                        auto val = [&](int j) { return fmaf(er, __uint_as_float(z[j]), __uint_as_float(y[j])); };
                        #pragma unroll
                        for (int j = 0; j < 4; j++)
                            if (c + 8 * j < vs)
                                *(uint4 *)(o + 8 * j) = make_uint4(pack_bf16(val(8 * j), val(8 * j + 1)), pack_bf16(val(8 * j + 2), val(8 * j + 3)),
                                                                   pack_bf16(val(8 * j + 4), val(8 * j + 5)), pack_bf16(val(8 * j + 6), val(8 * j + 7)));
                    }
                }
                asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                mbar_arrive(yfree + ((i - 1) & 1));
            }
            run_before = run;
        }
        if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 1024);
    }
    __syncthreads();
    if (warp == 13) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem), "r"(512) : "memory");
    }
}
