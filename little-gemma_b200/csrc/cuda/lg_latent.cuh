// lg_latent.cuh -- attention over a cache of latent rows.
//
// A layer caches ONE row per position, shared by all heads: [ latent c (kv_rank) | rotated key part (rot_dim) ].  Head h's
// unrotated key is W_uk[h] c and its value W_uv[h] c, so its score is  (q_h . W_uk[h] c + qrot_h . krot) * scale.
//
//  * decode / verify: the products are moved to the query side ("absorbed"): the query row [ W_uk[h]^T q_h | qrot_h ] meets the
//    cached rows directly, the attention output is a latent, and W_uv[h] is applied to it afterwards.  Every head reads the same
//    rows, so the heads of a token form the rows of one matrix product (lg_latent_dec_attn_kernel).
//  * prompt blocks: keys and values of the context are expanded per head by one wide matmul and the block runs an ordinary
//    causal attention with head sizes dim + rot_dim and vdim (lg_latent_pf_attn_kernel): far fewer operations per score.
//  * lg_latent_attn_rows_kernel: the absorbed form one (token, head) per CTA in f32 arithmetic, for 32-bit models and for sizes
//    the other kernels do not hold.
//
// A softmax has a sink: exp(sink_h) joins the denominator and has no value.
#pragma once
#include "lg_dense.cuh"

#define LG_LOG2E 1.4426950408889634f

__device__ __forceinline__ void split_bf16(float a, float b, uint32_t &hi, uint32_t &lo) {
    const bf16 ha = __float2bfloat16_rn(a), hb = __float2bfloat16_rn(b);
    hi = (uint32_t)__bfloat16_as_ushort(ha) | ((uint32_t)__bfloat16_as_ushort(hb) << 16);
    lo = pack_bf16(a - __bfloat162float(ha), b - __bfloat162float(hb));
}

// ---------------------------------------------------------------------------------------------
// one (token, head) per CTA, f32 arithmetic
// ---------------------------------------------------------------------------------------------
struct LgLatentRowsArgs {
    const void *q; const void *cache; int ldc, kvp;   // q: [tok * H + h][ldc]; cache: [position][ldc]; latent = the first kvp columns
    int H; const float *sink; float scale;
    const int *pos;
    void *out;                                        // [tok * H + h][kvp]
};
template <typename T>
__global__ void __launch_bounds__(128) lg_latent_attn_rows_kernel(LgLatentRowsArgs a) {
    extern __shared__ __align__(16) unsigned char lat_smem[];
    constexpr int S = 128;
    float *sq = (float *)lat_smem, *acc = sq + a.ldc, *sp = acc + a.kvp;
    __shared__ float red[32];
    pdl_launch(); pdl_wait();
    const int h = blockIdx.x, tok = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const size_t row = (size_t)tok * a.H + h;
    const T *q = (const T *)a.q + row * a.ldc, *cache = (const T *)a.cache;
    for (int i = threadIdx.x; i < a.ldc; i += blockDim.x) sq[i] = from_elem(q[i]);
    for (int i = threadIdx.x; i < a.kvp; i += blockDim.x) acc[i] = 0.0f;
    __syncthreads();
    const int n_keys = *a.pos + tok + 1;
    float m = a.sink[h] * LG_LOG2E, l = 1.0f;         // the sink is the first term of the denominator
    const float sc = a.scale * LG_LOG2E;
    for (int k0 = 0; k0 < n_keys; k0 += S) {
        const int nk = min(S, n_keys - k0);
        for (int k = warp; k < nk; k += 4) {
            const T *c = cache + (size_t)(k0 + k) * a.ldc;
            float d = 0.0f;
            for (int i = lane; i < a.ldc; i += 32) d = fmaf(sq[i], from_elem(c[i]), d);
            d = warp_sum(d);
            if (lane == 0) sp[k] = d * sc;
        }
        __syncthreads();
        const float s = threadIdx.x < nk ? sp[threadIdx.x] : -INFINITY;
        float mx = warp_max(s);
        if (lane == 0) red[warp] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float m_new = fmaxf(m, mx), alpha = exp2f(m - m_new), p = threadIdx.x < nk ? exp2f(s - m_new) : 0.0f;
        const float tot = block_sum(p, red);          // (its barriers order the reads of red and sp above before the writes below)
        if (threadIdx.x < nk) sp[threadIdx.x] = p;
        __syncthreads();
        l = l * alpha + tot; m = m_new;
        for (int i = threadIdx.x; i < a.kvp; i += blockDim.x) {
            float o = acc[i] * alpha;
            const T *c = cache + (size_t)k0 * a.ldc + i;
            for (int k = 0; k < nk; k++) o = fmaf(sp[k], from_elem(c[(size_t)k * a.ldc]), o);
            acc[i] = o;
        }
        __syncthreads();
    }
    for (int i = threadIdx.x; i < a.kvp; i += blockDim.x) to_elem(acc[i] / l, ((T *)a.out)[row * a.kvp + i]);
}

// the query rows of the absorbed form without a matmul to ride on (32-bit path)
template <typename T>
__global__ void lg_latent_rot_q_kernel(LgRotQ a) { pdl_launch(); pdl_wait(); rot_q_rows<T>(a, blockIdx.y, blockIdx.x * blockDim.x + threadIdx.x, gridDim.x * blockDim.x); }

// RMS-normed query latent rows and the block's cache rows, one CTA per token
struct LgLatentPrepArgs {
    const float *src; int ld, q_off, q_rank; const float *q_norm; float eps;
    void *cq; int ldcq;
    int owns; LgCacheRow cr;
};
template <typename T>
__global__ void __launch_bounds__(128) lg_latent_prep_kernel(LgLatentPrepArgs a) {
    __shared__ float red[32];
    pdl_launch(); pdl_wait();
    const int tok = blockIdx.x;
    const float *s = a.src + (size_t)tok * a.ld + a.q_off;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x) ss += s[i] * s[i];
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)a.q_rank + a.eps);
    for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x) to_elem(s[i] * inv * a.q_norm[i], ((T *)a.cq)[(size_t)tok * a.ldcq + i]);
    if (a.owns) cache_row<T>(a.cr, tok, red);
}

// ---------------------------------------------------------------------------------------------
// decode / verify: split over keys, all heads of the block's tokens as rows of one product
// ---------------------------------------------------------------------------------------------
// CTA (x, y): rows [16 RT y, 16 RT (y + 1)) of the M * H query rows; key tiles x, x + C, x + 2C, ... of 64 positions on absolute
// boundaries (C = gridDim.x comes from the cache length and the head count), online softmax over them, one partial (max, sum,
// latent row) per CTA and row.  A tile arrives by tiled TMA copies (blocks of 64 columns, 128-byte swizzle); the first one is
// requested before the dependency wait unless it holds rows of this very step.  Scores: warp (kg, kh) multiplies 16 keys x one
// half of the columns; the halves are added by the softmax.  Output: warp w owns NACC column groups of 8; the weights enter as
// bf16 high + low parts.  A row's arithmetic does not depend on the rows beside it.
#define LG_LD_S 64
#define LG_LD_THREADS 256
struct LgLatentDecArgs {
    const bf16 *q;                       // [M * H][ldc]
    int ldc, kvp;
    int rows, H;
    float scale; const int *pos;
    float *part; float2 *part_ml;        // [C][rows][kvp], [C][rows]
    int *err;
};
__host__ __device__ constexpr int lg_latent_blocks(int cols) { return (cols + 63) / 64; }
__host__ __device__ constexpr size_t lg_latent_dec_smem(int rt, int ldc) {
    return 1024 + (size_t)2 * lg_latent_blocks(ldc) * LG_LD_S * 128 + ((size_t)(rt * 16) * (ldc + 8) + (size_t)2 * rt * 16 * (LG_LD_S + 8)) * 2
         + ((size_t)2 * rt * 16 * (LG_LD_S + 4) + (size_t)3 * rt * 16) * 4 + 16;
}
template <int RT, int NACC>
__global__ void __launch_bounds__(LG_LD_THREADS, 1) lg_latent_dec_attn_kernel(const __grid_constant__ CUtensorMap tmc, LgLatentDecArgs a) {
    extern __shared__ __align__(16) unsigned char lat_smem[];
    constexpr int R = RT * 16, S = LG_LD_S, LP = S + 8, LS = S + 4;
    const int lq = a.ldc + 8, nblk = lg_latent_blocks(a.ldc), tile_bytes = nblk * S * 128;
    unsigned char *sK = (unsigned char *)(((uintptr_t)lat_smem + 1023) & ~(uintptr_t)1023);
    bf16 *sQ = (bf16 *)(sK + 2 * tile_bytes), *sPh = sQ + (size_t)R * lq, *sPl = sPh + R * LP;
    float *sS = (float *)(sPl + R * LP), *sM = sS + 2 * R * LS, *sL = sM + R, *sA = sL + R;
    uint64_t *full = (uint64_t *)(sA + R);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int row0 = blockIdx.y * R, C = gridDim.x;
    pdl_launch();
    // the position and every row below it come from earlier forwards
    const int pos = *a.pos;
    const int last_row = min(row0 + R, a.rows) - 1;
    const int n_keys = pos + last_row / a.H + 1;                   // keys the last token of this CTA's rows sees
    const int n_tiles = (n_keys + S - 1) / S;
    if ((int)blockIdx.x >= n_tiles) return;
    auto load_tile = [&](int tile, int buf) {                      // thread 0
        mbar_expect_tx(full + buf, tile_bytes);
        for (int i = 0; i < nblk; i++) tma_load_2d(sK + buf * tile_bytes + i * S * 128, &tmc, i * 64, tile * S, full + buf);
    };
    const bool early = ((int)blockIdx.x + 1) * S <= pos;
    if (tid == 0) {
        mbar_init(full, 1); mbar_init(full + 1, 1);
        if (early) load_tile(blockIdx.x, 0);
    }
    if (tid < R) { sM[tid] = -INFINITY; sL[tid] = 0.0f; }
    pdl_wait();
    if (tid == 0 && !early) load_tile(blockIdx.x, 0);
    const int cpr = a.ldc >> 3;                                    // 16-byte chunks per query row
    for (int r = warp; r < R; r += LG_LD_THREADS / 32)
        for (int c = lane; c < cpr; c += 32)
            *(uint4 *)(sQ + (size_t)r * lq + c * 8) = row0 + r < a.rows ? *(const uint4 *)(a.q + (size_t)(row0 + r) * a.ldc + c * 8) : make_uint4(0, 0, 0, 0);
    float acc[RT][NACC][4];
    #pragma unroll
    for (int r = 0; r < RT; r++)
        #pragma unroll
        for (int n = 0; n < NACC; n++)
            #pragma unroll
            for (int i = 0; i < 4; i++) acc[r][n][i] = 0.0f;
    const int col0 = warp * NACC * 8;
    const int kg = warp & 3, kh = warp >> 2, nk16 = a.ldc >> 4, ks_lo = kh ? nk16 >> 1 : 0, ks_hi = kh ? nk16 : nk16 >> 1;
    const float sc = a.scale * LG_LOG2E;
    const int qr = (lane & 7) + ((lane >> 3) & 1) * 8, qc = ((lane >> 4) & 1) * 8;               // this lane's row / column of a 16 x 16 A block
    const int kr = kg * 16 + (lane & 7) + ((lane >> 4) & 1) * 8, kc = (lane >> 3) & 1;           // key row and 8-column half of a B block
    const int x7 = lane & 7;                                                                     // a row's chunks are permuted by row % 8
    __syncthreads();
    uint32_t ph = 0;
    int buf = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < n_tiles; tile += C, buf ^= 1) {
        if (tid == 0 && tile + C < n_tiles) load_tile(tile + C, buf ^ 1);
        if (ok && !mbar_wait(full + buf, (ph >> buf) & 1)) { ok = false; if (lane == 0) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT); }
        ph ^= 1u << buf;
        const unsigned char *K = sK + buf * tile_bytes;
        {   // scores of 16 keys over this warp's half of the columns
            float s[RT][2][4];
            #pragma unroll
            for (int r = 0; r < RT; r++)
                #pragma unroll
                for (int n = 0; n < 2; n++)
                    #pragma unroll
                    for (int i = 0; i < 4; i++) s[r][n][i] = 0.0f;
            const unsigned char *kp = K + kr * 128;
            const bf16 *qp = sQ + (size_t)qr * lq + qc;
            #pragma unroll 4
            for (int kk = ks_lo; kk < ks_hi; kk++) {
                uint32_t b[4];
                ldsm_x4(b, kp + (kk >> 2) * (S * 128) + ((((kk & 3) * 2 + kc) ^ x7) << 4));
                #pragma unroll
                for (int r = 0; r < RT; r++) {
                    uint32_t q4[4];
                    ldsm_x4(q4, qp + (size_t)r * 16 * lq + kk * 16);
                    mma_bf16(s[r][0], q4[0], q4[1], q4[2], q4[3], b[0], b[1]);
                    mma_bf16(s[r][1], q4[0], q4[1], q4[2], q4[3], b[2], b[3]);
                }
            }
            #pragma unroll
            for (int r = 0; r < RT; r++)
                #pragma unroll
                for (int n = 0; n < 2; n++) {
                    float *d = sS + (size_t)kh * R * LS + (size_t)(r * 16 + g) * LS + kg * 16 + n * 8 + 2 * t;
                    *(float2 *)d = make_float2(s[r][n][0], s[r][n][1]);
                    *(float2 *)(d + 8 * LS) = make_float2(s[r][n][2], s[r][n][3]);
                }
        }
        __syncthreads();
        #pragma unroll
        for (int rr = 0; rr < RT * 2; rr++) {          // softmax: a warp per row, two keys per lane
            const int r = warp * RT * 2 + rr, row = row0 + r;
            const float2 s0 = *(const float2 *)(sS + (size_t)r * LS + 2 * lane), s1 = *(const float2 *)(sS + (size_t)(R + r) * LS + 2 * lane);
            const int key = tile * S + 2 * lane, seen = row < a.rows ? pos + row / a.H : -1;
            const float v0 = key <= seen ? (s0.x + s1.x) * sc : -INFINITY, v1 = key + 1 <= seen ? (s0.y + s1.y) * sc : -INFINITY;
            const float m_old = sM[r], m_new = fmaxf(m_old, warp_max(fmaxf(v0, v1)));
            const float p0 = m_new == -INFINITY ? 0.0f : exp2f(v0 - m_new), p1 = m_new == -INFINITY ? 0.0f : exp2f(v1 - m_new);
            const float sum = warp_sum(p0 + p1);
            uint32_t hi, lo;
            split_bf16(p0, p1, hi, lo);
            *(uint32_t *)(sPh + r * LP + 2 * lane) = hi;
            *(uint32_t *)(sPl + r * LP + 2 * lane) = lo;
            if (lane == 0) {
                const float al = m_old == -INFINITY ? 0.0f : exp2f(m_old - m_new);
                sA[r] = al; sM[r] = m_new; sL[r] = sL[r] * al + sum;
            }
        }
        __syncthreads();
        if (col0 < a.kvp) {
            #pragma unroll
            for (int r = 0; r < RT; r++) {
                const float a0 = sA[r * 16 + g], a1 = sA[r * 16 + g + 8];
                #pragma unroll
                for (int n = 0; n < NACC; n++) { acc[r][n][0] *= a0; acc[r][n][1] *= a0; acc[r][n][2] *= a1; acc[r][n][3] *= a1; }
            }
            const unsigned char *vp = K + qr * 128;
            const int po = qr * LP + qc;
            #pragma unroll
            for (int k16 = 0; k16 < S / 16; k16++) {
                uint32_t p4h[RT][4], p4l[RT][4];
                #pragma unroll
                for (int r = 0; r < RT; r++) { ldsm_x4(p4h[r], sPh + r * 16 * LP + po + k16 * 16); ldsm_x4(p4l[r], sPl + r * 16 * LP + po + k16 * 16); }
                #pragma unroll
                for (int n = 0; n < NACC; n += 2) {
                    const int c8 = (col0 >> 3) + n;                      // 8-column group
                    if (c8 * 8 >= a.kvp) break;
                    uint32_t v[4];
                    ldsm_x4_t(v, vp + k16 * 16 * 128 + (c8 >> 3) * (S * 128) + ((((c8 & 7) + (qc >> 3)) ^ x7) << 4));
                    #pragma unroll
                    for (int r = 0; r < RT; r++) {
                        mma_bf16(acc[r][n], p4h[r][0], p4h[r][1], p4h[r][2], p4h[r][3], v[0], v[1]);
                        mma_bf16(acc[r][n + 1], p4h[r][0], p4h[r][1], p4h[r][2], p4h[r][3], v[2], v[3]);
                        mma_bf16(acc[r][n], p4l[r][0], p4l[r][1], p4l[r][2], p4l[r][3], v[0], v[1]);
                        mma_bf16(acc[r][n + 1], p4l[r][0], p4l[r][1], p4l[r][2], p4l[r][3], v[2], v[3]);
                    }
                }
            }
        }
        __syncthreads();                               // the tile's buffer is free for the copy after next
    }
    #pragma unroll
    for (int r = 0; r < RT; r++)
        #pragma unroll
        for (int n = 0; n < NACC; n++) {
            const int col = col0 + n * 8 + 2 * t, r_lo = row0 + r * 16 + g;
            if (col >= a.kvp) continue;
            float *o = a.part + ((size_t)blockIdx.x * a.rows + r_lo) * a.kvp + col;
            if (r_lo < a.rows) *(float2 *)o = make_float2(acc[r][n][0], acc[r][n][1]);
            if (r_lo + 8 < a.rows) *(float2 *)(o + (size_t)8 * a.kvp) = make_float2(acc[r][n][2], acc[r][n][3]);
        }
    if (tid < R && row0 + tid < a.rows) a.part_ml[(size_t)blockIdx.x * a.rows + row0 + tid] = make_float2(sM[tid], sL[tid]);
}

// Merge of the partials with the sink: latent output rows in bf16.  One CTA per query row; group g of its threads takes splits
// g, g + GROUPS, ..., the first LG_LM_PRE of them loaded while the weights are still being made.
struct LgLatentMergeArgs {
    const float *part; const float2 *part_ml; int rows, H, kvp, C;
    const float *sink; const int *pos;
    bf16 *out;                           // [rows][kvp]
};
#define LG_LM_GROUPS 8
#define LG_LM_THREADS 1024
#define LG_LM_PRE 4
#define LG_LM_MAXC 160
__global__ void __launch_bounds__(LG_LM_THREADS) lg_latent_merge_kernel(LgLatentMergeArgs a) {
    extern __shared__ __align__(16) unsigned char lat_smem[];
    float *sum = (float *)lat_smem;                    // [groups][kvp]
    __shared__ float w[LG_LM_MAXC];
    __shared__ float s_inv;
    pdl_launch();
    const int row = blockIdx.x, tid = threadIdx.x, lane = tid & 31;
    const int n = min(a.C, (*a.pos + row / a.H + LG_LD_S) / LG_LD_S);            // splits that hold keys of this row
    const float sink = a.sink[row % a.H] * LG_LOG2E;
    constexpr int TPG = LG_LM_THREADS / LG_LM_GROUPS;
    const int grp = tid / TPG, ti = tid % TPG;
    pdl_wait();
    const float *part = a.part + (size_t)row * a.kvp;
    const size_t stride = (size_t)a.rows * a.kvp;
    float4 v[LG_LM_PRE];
    #pragma unroll
    for (int j = 0; j < LG_LM_PRE; j++) {
        const int i = grp + j * LG_LM_GROUPS;
        v[j] = i < n && ti * 4 < a.kvp ? *(const float4 *)(part + i * stride + ti * 4) : make_float4(0, 0, 0, 0);
    }
    if (tid < 32) {
        float m = sink;
        for (int i = lane; i < n; i += 32) m = fmaxf(m, a.part_ml[(size_t)i * a.rows + row].x);
        m = warp_max(m);
        float l = lane == 0 ? exp2f(sink - m) : 0.0f;
        for (int i = lane; i < n; i += 32) {
            const float2 ml = a.part_ml[(size_t)i * a.rows + row];
            const float e = ml.x == -INFINITY ? 0.0f : exp2f(ml.x - m);
            w[i] = e;
            l += ml.y * e;
        }
        l = warp_sum(l);
        if (lane == 0) s_inv = 1.0f / l;
    }
    __syncthreads();
    for (int c = ti * 4; c < a.kvp; c += TPG * 4) {
        float4 o = make_float4(0, 0, 0, 0);
        auto add = [&](int i, const float4 &x) { const float wi = w[i]; o.x = fmaf(wi, x.x, o.x); o.y = fmaf(wi, x.y, o.y); o.z = fmaf(wi, x.z, o.z); o.w = fmaf(wi, x.w, o.w); };
        int i0 = grp;
        if (c == ti * 4) {
            #pragma unroll
            for (int j = 0; j < LG_LM_PRE; j++, i0 += LG_LM_GROUPS) if (i0 < n) add(i0, v[j]);
        }
        #pragma unroll 4
        for (int i = i0; i < n; i += LG_LM_GROUPS) add(i, *(const float4 *)(part + i * stride + c));
        *(float4 *)(sum + (size_t)grp * a.kvp + c) = o;
    }
    __syncthreads();
    const float inv = s_inv;
    for (int c = tid; c < a.kvp; c += LG_LM_THREADS) {
        float o = 0.0f;
        #pragma unroll
        for (int i = 0; i < LG_LM_GROUPS; i++) o += sum[(size_t)i * a.kvp + c];
        a.out[(size_t)row * a.kvp + c] = __float2bfloat16_rn(o * inv);
    }
}

// ---------------------------------------------------------------------------------------------
// prompt blocks: causal attention over expanded keys and values, on tcgen05
// ---------------------------------------------------------------------------------------------
// CTA = one head x 128 query rows (the TMEM lanes), key tiles of 64.  Keys come as [key][H dimp] (expanded) plus the rotated
// part of the cache rows, values transposed as [H vdp][key], queries already rotated; every operand is K-major in blocks of 64
// columns (128-byte swizzle) loaded by tiled TMA copies.
//   warp 4 (one thread)  Q once, then K tiles;   warp 6 (one thread)  V tiles;
//   warp 5 (one thread)  tcgen05.mma: S(i + 1) = Q K^T into one of two 64-column buffers while tile i is in its softmax, then
//                        O += P(i) V with P read from tensor memory;
//   warps 0-3            one query row per thread: S from tensor memory, online softmax in f32, P back over S's columns as bf16
//                        high + low parts.  O is rescaled only when a row's maximum has grown by more than 2^LG_LP_SLACK since
//                        the maximum in use -- until then the weights are merely larger than 1 -- which needs the previous
//                        product to have finished.
//   The rows can be two tiles ahead of the products, so the weights' and the products' barriers exist once per buffer: of one barrier for both,
//   a parity could stand for the phase before or after the one that is waited for.
// The softmax starts from the sink: maximum = sink, sum = 1.  The output gate is applied to the finished rows.
#define LG_LP_Q 128
#define LG_LP_S 64
#define LG_LP_THREADS 224
#define LG_LP_SLACK 8.0f
struct LgLatentPfArgs {
    int H, dimp, rotp, vdp, n, rot_at;
    float scale; const float *sink;
    const float *gate; int ldg;          // [tok][H vdp]
    const int *pos;
    bf16 *out; int ldo;                  // [tok][H vdp]
    int *err;
};
__host__ __device__ constexpr size_t lg_latent_pf_smem(int dimp, int rotp, int vdp) {
    return 1024 + (size_t)(lg_latent_blocks(dimp) + lg_latent_blocks(rotp)) * (LG_LP_Q + LG_LP_S) * 128 + (size_t)vdp * 128 + 128;
}
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&r)[32]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
                 "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};"
                 :: "r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
                    "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
                    "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
                    "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31]) : "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
                 :: "r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
                    "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
__device__ __forceinline__ void tmem_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// the A operand from tensor memory: lane = row, two 16-bit elements of k per column
__device__ __forceinline__ void umma_f16_ta(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
                 :: "r"(d_tmem), "r"(a_tmem), "l"(bdesc), "r"(idesc), "r"(accumulate) : "memory");
}

// the rotated part of every head's query, in place (the wide pass)
__global__ void lg_latent_rot_rows_kernel(LgRotQ a) { pdl_launch(); pdl_wait(); rot_q_in_place(a, blockIdx.y, blockIdx.x * blockDim.x + threadIdx.x, gridDim.x * blockDim.x); }

__global__ void __launch_bounds__(LG_LP_THREADS, 2)
lg_latent_pf_attn_kernel(const __grid_constant__ CUtensorMap tmq, const __grid_constant__ CUtensorMap tmk, const __grid_constant__ CUtensorMap tmr,
                         const __grid_constant__ CUtensorMap tmv, LgLatentPfArgs a) {
    extern __shared__ __align__(16) unsigned char lat_smem[];
    constexpr int Q_BYTES = LG_LP_Q * 128, K_BYTES = LG_LP_S * 128;
    const int kb = lg_latent_blocks(a.dimp), nb = kb + lg_latent_blocks(a.rotp), dq = a.dimp + a.rotp;
    unsigned char *sQ = (unsigned char *)(((uintptr_t)lat_smem + 1023) & ~(uintptr_t)1023), *sK = sQ + nb * Q_BYTES, *sV = sK + nb * K_BYTES;
    uint64_t *qfull = (uint64_t *)(sV + (size_t)a.vdp * 128), *kfull = qfull + 1, *kempty = qfull + 2, *vfull = qfull + 3, *vempty = qfull + 4,
             *sfull = qfull + 5 /* two */, *pready = qfull + 7 /* two */, *odone = qfull + 9 /* two */;
    uint32_t *tmem_slot = (uint32_t *)(qfull + 11);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y, qb = (gridDim.x - 1 - blockIdx.x) * LG_LP_Q;       // longest rows first
    const uint32_t tcols = a.vdp <= 128 ? 256 : 512;                             // S / P twice 64 columns, O vdp columns

    if (threadIdx.x == 0) {
        mbar_init(qfull, 1); mbar_init(kfull, 1); mbar_init(kempty, 1); mbar_init(vfull, 1); mbar_init(vempty, 1);
        mbar_init(sfull, 1); mbar_init(sfull + 1, 1); mbar_init(pready, 128); mbar_init(pready + 1, 128); mbar_init(odone, 1); mbar_init(odone + 1, 1);
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(smem_u32(tmem_slot)), "r"(tcols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot, tO = tmem + 2 * LG_LP_S;
    pdl_launch();                        // only now: a dependant must not take tensor memory a CTA of this grid still waits for
    pdl_wait();
    const int pos = *a.pos;
    const int n_tiles = (pos + min(qb + LG_LP_Q, a.n) + LG_LP_S - 1) / LG_LP_S;

    if (warp == 4) {
        if (lane == 0) {
            mbar_expect_tx(qfull, nb * Q_BYTES);
            for (int c = 0; c < nb; c++) tma_load_2d(sQ + c * Q_BYTES, &tmq, h * dq + (c < kb ? c * 64 : a.dimp + (c - kb) * 64), qb, qfull);
            int i = 0;
            for (; i < n_tiles; i++) {
                if (i && !mbar_wait(kempty, (i - 1) & 1)) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 4); break; }
                mbar_expect_tx(kfull, nb * K_BYTES);
                for (int c = 0; c < nb; c++) {
                    if (c < kb) tma_load_2d(sK + c * K_BYTES, &tmk, h * a.dimp + c * 64, i * LG_LP_S, kfull);
                    else tma_load_2d(sK + c * K_BYTES, &tmr, a.rot_at + (c - kb) * 64, i * LG_LP_S, kfull);
                }
            }
            if (i < n_tiles) { mbar_wait(qfull, 0); if (i) mbar_wait(kfull, (i - 1) & 1); }      // own copies in flight land before the CTA ends
        }
    } else if (warp == 6) {
        if (lane == 0) {
            int i = 0;
            for (; i < n_tiles; i++) {
                if (i && !mbar_wait(vempty, (i - 1) & 1)) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 16); break; }
                mbar_expect_tx(vfull, a.vdp * 128);
                tma_load_2d(sV, &tmv, i * LG_LP_S, h * a.vdp, vfull);
            }
            if (i < n_tiles && i) mbar_wait(vfull, (i - 1) & 1);
        }
    } else if (warp == 5) {
        if (lane == 0) {
            // f32 accumulator, bf16 x bf16, K-major; N = keys of a tile / value columns
            const uint32_t fmt = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(LG_LP_Q >> 4) << 24);
            const uint32_t idS = fmt | ((uint32_t)(LG_LP_S >> 3) << 17), idO = fmt | ((uint32_t)(a.vdp >> 3) << 17);
            const uint64_t qd = umma_desc_k128(smem_u32(sQ)), kd = umma_desc_k128(smem_u32(sK)), vd = umma_desc_k128(smem_u32(sV));
            bool ok = mbar_wait(qfull, 0);
            auto scores = [&](int i) {
                if (!mbar_wait(kfull, i & 1)) return false;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t tS = tmem + (i & 1) * LG_LP_S;
                uint32_t acc = 0;
                for (int c = 0; c < nb; c++) {
                    const int left = c < kb ? a.dimp - c * 64 : a.rotp - (c - kb) * 64, steps = min(left, 64) >> 4;
                    for (int j = 0; j < steps; j++) { umma_f16(tS, qd + c * (Q_BYTES >> 4) + 2 * j, kd + c * (K_BYTES >> 4) + 2 * j, idS, acc); acc = 1; }
                }
                umma_commit(kempty);
                umma_commit(sfull + (i & 1));
                return true;
            };
            ok = ok && scores(0);
            for (int i = 0; i < n_tiles && ok; i++) {
                if (i + 1 < n_tiles) ok = scores(i + 1);
                ok = ok && mbar_wait(pready + (i & 1), (i >> 1) & 1) && mbar_wait(vfull, i & 1);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t tP = tmem + (i & 1) * LG_LP_S;
                #pragma unroll
                for (int j = 0; j < 4; j++) umma_f16_ta(tO, tP + 8 * j, vd + 2 * j, idO, (i | j) ? 1u : 0u);
                #pragma unroll
                for (int j = 0; j < 4; j++) umma_f16_ta(tO, tP + 32 + 8 * j, vd + 2 * j, idO, 1u);
                umma_commit(vempty);
                umma_commit(odone + (i & 1));
            }
            if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 8);
        }
    } else {
        const int tok = qb + threadIdx.x, q_pos = pos + tok;
        const uint32_t lanes = (uint32_t)(warp * 32) << 16;
        const float sc = a.scale * LG_LOG2E, sink = a.sink[h] * LG_LOG2E;
        const int first_edge = (pos + qb + warp * 32 + 1) / LG_LP_S;               // tiles below it are seen whole by every row of the warp
        float m = sink, l = 1.0f;
        bool ok = true;
        for (int i = 0; i < n_tiles; i++) {
            ok = __all_sync(0xffffffffu, mbar_wait(sfull + (i & 1), (i >> 1) & 1));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t tS = tmem + lanes + (i & 1) * LG_LP_S;
            uint32_t s0[32], s1[32];
            __syncwarp();
            tmem_ld32(tS, s0);
            tmem_ld32(tS + 32, s1);
            float mx = -INFINITY;
            #pragma unroll
            for (int j = 0; j < 32; j++) {
                if (i >= first_edge) {
                    const int key = i * LG_LP_S + j;
                    if (key > q_pos) s0[j] = 0xff800000u;
                    if (key + 32 > q_pos) s1[j] = 0xff800000u;
                }
                mx = fmaxf(mx, fmaxf(__uint_as_float(s0[j]), __uint_as_float(s1[j])));
            }
            // a row's scores are scaled once more in the exponent: exp2(s * sc - m)
            const float mt = mx * sc;
            const bool grow = i == 0 || mt > m + LG_LP_SLACK;
            if (__any_sync(0xffffffffu, grow)) {
                const float m_new = fmaxf(m, mt), alpha = exp2f(m - m_new);
                if (i) {
                    ok = __all_sync(0xffffffffu, mbar_wait(odone + ((i - 1) & 1), ((i - 1) >> 1) & 1));
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    for (int c = 0; c < a.vdp; c += 32) {
                        uint32_t o[32];
                        __syncwarp();
                        tmem_ld32(tO + lanes + c, o);
                        #pragma unroll
                        for (int j = 0; j < 32; j++) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
                        tmem_st32(tO + lanes + c, o);
                    }
                    tmem_wait_st();
                }
                l *= alpha; m = m_new;
            }
            #pragma unroll
            for (int half = 0; half < 2; half++) {
                uint32_t hi[16], lo[16];
                #pragma unroll
                for (int j = 0; j < 16; j++) {
                    const float x = __uint_as_float(half ? s1[2 * j] : s0[2 * j]), y = __uint_as_float(half ? s1[2 * j + 1] : s0[2 * j + 1]);
                    const float p = ex2(fmaf(x, sc, -m)), q = ex2(fmaf(y, sc, -m));
                    l += p + q;
                    split_bf16(p, q, hi[j], lo[j]);
                }
                __syncwarp();
                tmem_st16(tS + 16 * half, hi);
                tmem_st16(tS + 32 + 16 * half, lo);
            }
            tmem_wait_st();
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(pready + (i & 1));       // (a barrier per buffer: both tiles' weights may be ready before the products ask for the first)
        }
        ok = __all_sync(0xffffffffu, ok && mbar_wait(odone + ((n_tiles - 1) & 1), ((n_tiles - 1) >> 1) & 1));
        if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 32);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const float inv = 1.0f / l;
        if (ok)
            for (int c = 0; c < a.vdp; c += 32) {
                uint32_t o[32];
                __syncwarp();
                tmem_ld32(tO + lanes + c, o);
                if (tok >= a.n) continue;
                const float4 *gt = (const float4 *)(a.gate + (size_t)tok * a.ldg + h * a.vdp + c);
                uint4 *dst = (uint4 *)(a.out + (size_t)tok * a.ldo + h * a.vdp + c);
                #pragma unroll
                for (int j = 0; j < 4; j++) {
                    if (c + j * 8 >= a.vdp) break;
                    const float4 g0 = gt[2 * j], g1 = gt[2 * j + 1];
                    auto val = [&](int k, float gg) { return __uint_as_float(o[8 * j + k]) * inv * sigmoid_f(gg); };
                    dst[j] = make_uint4(pack_bf16(val(0, g0.x), val(1, g0.y)), pack_bf16(val(2, g0.z), val(3, g0.w)),
                                        pack_bf16(val(4, g1.x), val(5, g1.y)), pack_bf16(val(6, g1.z), val(7, g1.w)));
                }
            }
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    }
    __syncthreads();
    if (warp == 5) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem), "r"(tcols) : "memory");
    }
}
