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

__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" :: "n"(N) : "memory"); }
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
// latent row) per CTA and row.  Scores: warp (kg, kh) multiplies 16 keys x one half of the columns; the halves are added by the
// softmax.  Output: warp w owns NACC column groups of 8; the weights enter as bf16 high + low parts.  A row's arithmetic does
// not depend on the rows beside it.
#define LG_LD_S 64
#define LG_LD_THREADS 256
struct LgLatentDecArgs {
    const bf16 *q;                       // [M * H][ldc]
    const bf16 *cache; int ldc, kvp;
    int rows, H;
    float scale; const int *pos;
    float *part; float2 *part_ml;        // [C][rows][kvp], [C][rows]
};
__host__ __device__ constexpr size_t lg_latent_dec_smem(int rt, int ldc) {
    return ((size_t)(rt * 16) * (ldc + 8) + (size_t)2 * LG_LD_S * (ldc + 8) + (size_t)2 * rt * 16 * (LG_LD_S + 8)) * 2
         + ((size_t)2 * rt * 16 * (LG_LD_S + 4) + (size_t)3 * rt * 16) * 4;
}
template <int RT, int NACC>
__global__ void __launch_bounds__(LG_LD_THREADS, 1) lg_latent_dec_attn_kernel(LgLatentDecArgs a) {
    extern __shared__ __align__(16) unsigned char lat_smem[];
    constexpr int R = RT * 16, S = LG_LD_S, LP = S + 8, LS = S + 4;
    const int lq = a.ldc + 8;
    bf16 *sQ = (bf16 *)lat_smem, *sK = sQ + (size_t)R * lq, *sPh = sK + (size_t)2 * S * lq, *sPl = sPh + R * LP;
    float *sS = (float *)(sPl + R * LP), *sM = sS + 2 * R * LS, *sL = sM + R, *sA = sL + R;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int row0 = blockIdx.y * R, C = gridDim.x;
    pdl_launch(); pdl_wait();
    const int pos = *a.pos;
    const int last_row = min(row0 + R, a.rows) - 1;
    const int n_keys = pos + last_row / a.H + 1;                   // keys the last token of this CTA's rows sees
    const int n_tiles = (n_keys + S - 1) / S;
    if ((int)blockIdx.x >= n_tiles) return;

    const int cpr = a.ldc >> 3;                                    // 16-byte chunks per row
    auto load_tile = [&](int tile, int buf) {
        const bf16 *src = a.cache + (size_t)tile * S * a.ldc;
        bf16 *dst = sK + (size_t)buf * S * lq;
        const int valid = min(S, n_keys - tile * S);
        for (int u = tid; u < S * cpr; u += LG_LD_THREADS) {
            const int r = u / cpr, c = u % cpr;
            if (r < valid) cp_async16(dst + (size_t)r * lq + c * 8, src + (size_t)r * a.ldc + c * 8);
            else *(uint4 *)(dst + (size_t)r * lq + c * 8) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    };
    for (int u = tid; u < R * cpr; u += LG_LD_THREADS) {
        const int r = u / cpr, c = u % cpr;
        if (row0 + r < a.rows) cp_async16(sQ + (size_t)r * lq + c * 8, a.q + (size_t)(row0 + r) * a.ldc + c * 8);
        else *(uint4 *)(sQ + (size_t)r * lq + c * 8) = make_uint4(0, 0, 0, 0);
    }
    load_tile(blockIdx.x, 0);
    if (tid < R) { sM[tid] = -INFINITY; sL[tid] = 0.0f; }
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
    int buf = 0;
    for (int tile = blockIdx.x; tile < n_tiles; tile += C, buf ^= 1) {
        if (tile + C < n_tiles) { load_tile(tile + C, buf ^ 1); cp_async_wait<1>(); } else cp_async_wait<0>();
        __syncthreads();
        const bf16 *K = sK + (size_t)buf * S * lq;
        {   // scores of 16 keys over this warp's half of the columns
            float s[RT][2][4];
            #pragma unroll
            for (int r = 0; r < RT; r++)
                #pragma unroll
                for (int n = 0; n < 2; n++)
                    #pragma unroll
                    for (int i = 0; i < 4; i++) s[r][n][i] = 0.0f;
            const bf16 *kp = K + (size_t)(kg * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * lq + ((lane >> 3) & 1) * 8;
            const bf16 *qp = sQ + (size_t)((lane & 7) + ((lane >> 3) & 1) * 8) * lq + ((lane >> 4) & 1) * 8;
            #pragma unroll 4
            for (int kk = ks_lo; kk < ks_hi; kk++) {
                uint32_t b[4];
                ldsm_x4(b, kp + kk * 16);
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
            const bf16 *vp = K + (size_t)((lane & 7) + ((lane >> 3) & 1) * 8) * lq + col0 + ((lane >> 4) & 1) * 8;
            const int po = ((lane & 7) + ((lane >> 3) & 1) * 8) * LP + ((lane >> 4) & 1) * 8;
            #pragma unroll
            for (int k16 = 0; k16 < S / 16; k16++) {
                uint32_t ph[RT][4], pl[RT][4];
                #pragma unroll
                for (int r = 0; r < RT; r++) { ldsm_x4(ph[r], sPh + r * 16 * LP + po + k16 * 16); ldsm_x4(pl[r], sPl + r * 16 * LP + po + k16 * 16); }
                #pragma unroll
                for (int n = 0; n < NACC; n += 2) {
                    if (col0 + n * 8 >= a.kvp) break;
                    uint32_t v[4];
                    ldsm_x4_t(v, vp + (size_t)k16 * 16 * lq + n * 8);
                    #pragma unroll
                    for (int r = 0; r < RT; r++) {
                        mma_bf16(acc[r][n], ph[r][0], ph[r][1], ph[r][2], ph[r][3], v[0], v[1]);
                        mma_bf16(acc[r][n], pl[r][0], pl[r][1], pl[r][2], pl[r][3], v[0], v[1]);
                        mma_bf16(acc[r][n + 1], ph[r][0], ph[r][1], ph[r][2], ph[r][3], v[2], v[3]);
                        mma_bf16(acc[r][n + 1], pl[r][0], pl[r][1], pl[r][2], pl[r][3], v[2], v[3]);
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

// Merge of the partials, in ascending split order, with the sink: latent output rows in bf16.  One CTA per query row; four
// groups of threads take every fourth split.
struct LgLatentMergeArgs {
    const float *part; const float2 *part_ml; int rows, H, kvp, C;
    const float *sink; const int *pos;
    bf16 *out;                           // [rows][kvp]
};
#define LG_LM_GROUPS 4
#define LG_LM_THREADS 512
#define LG_LM_MAXC 160
__global__ void __launch_bounds__(LG_LM_THREADS) lg_latent_merge_kernel(LgLatentMergeArgs a) {
    extern __shared__ __align__(16) unsigned char lat_smem[];
    float *sum = (float *)lat_smem;                    // [groups][kvp]
    __shared__ float w[LG_LM_MAXC];
    __shared__ float red[32];
    pdl_launch(); pdl_wait();
    const int row = blockIdx.x, tid = threadIdx.x, lane = tid & 31;
    const int n = min(a.C, (*a.pos + row / a.H + LG_LD_S) / LG_LD_S);            // splits that hold keys of this row
    const float sink = a.sink[row % a.H] * LG_LOG2E;
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
        if (lane == 0) red[0] = 1.0f / l;
    }
    __syncthreads();
    const float inv = red[0];
    const int grp = tid / (LG_LM_THREADS / LG_LM_GROUPS), ti = tid % (LG_LM_THREADS / LG_LM_GROUPS);
    for (int c = ti * 4; c < a.kvp; c += LG_LM_THREADS / LG_LM_GROUPS * 4) {
        float4 o = make_float4(0, 0, 0, 0);
        #pragma unroll 4
        for (int i = grp; i < n; i += LG_LM_GROUPS) {
            const float4 v = *(const float4 *)(a.part + ((size_t)i * a.rows + row) * a.kvp + c);
            const float wi = w[i];
            o.x = fmaf(wi, v.x, o.x); o.y = fmaf(wi, v.y, o.y); o.z = fmaf(wi, v.z, o.z); o.w = fmaf(wi, v.w, o.w);
        }
        *(float4 *)(sum + (size_t)grp * a.kvp + c) = o;
    }
    __syncthreads();
    for (int c = tid; c < a.kvp; c += LG_LM_THREADS) {
        float v = 0.0f;
        #pragma unroll
        for (int i = 0; i < LG_LM_GROUPS; i++) v += sum[(size_t)i * a.kvp + c];
        a.out[(size_t)row * a.kvp + c] = __float2bfloat16_rn(v * inv);
    }
}

// ---------------------------------------------------------------------------------------------
// prompt blocks: causal attention over expanded keys and values
// ---------------------------------------------------------------------------------------------
// CTA = one head x 128 query rows (8 warps x 16), online softmax over key tiles of 64 (double-buffered cp.async).  A key row is
// its head's expanded part (dimp columns of `ex`) followed by the cache row's rotated part.  Queries are rotated as they are
// loaded.  The weights enter the second product as bf16 high + low parts; the output gate is applied to the finished rows.
#define LG_LP_Q 128
#define LG_LP_S 64
#define LG_LP_THREADS 256
struct LgLatentPfArgs {
    const bf16 *q; int ldq;              // [tok][H][dimp + rotp]
    const bf16 *ex; int ldx;             // [key][H dimp | H vdp]
    const bf16 *cache; int ldc, rot_at;
    int H, dimp, rotp, rot_dims, vdp, n;
    const float2 *tab; const float *sink; float scale;
    const float *gate; int ldg;          // [tok][H vdp]
    const int *pos;
    bf16 *out; int ldo;                  // [tok][H vdp]
};
__host__ __device__ constexpr size_t lg_latent_pf_smem(int dq, int vdp) {
    return ((size_t)LG_LP_Q * (dq + 8) + (size_t)2 * LG_LP_S * (dq + 8) + (size_t)2 * LG_LP_S * (vdp + 8)) * 2;
}
template <int NV>                        // value columns / 8, at most
__global__ void __launch_bounds__(LG_LP_THREADS, 1) lg_latent_pf_attn_kernel(LgLatentPfArgs a) {
    extern __shared__ __align__(16) unsigned char lat_smem[];
    const int dq = a.dimp + a.rotp, lq = dq + 8, lv = a.vdp + 8;
    bf16 *sQ = (bf16 *)lat_smem, *sK = sQ + (size_t)LG_LP_Q * lq, *sV = sK + (size_t)2 * LG_LP_S * lq;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.y, qb = (gridDim.x - 1 - blockIdx.x) * LG_LP_Q;       // longest rows first
    pdl_launch(); pdl_wait();
    const int pos = *a.pos;
    const int n_keys = pos + min(qb + LG_LP_Q, a.n), n_tiles = (n_keys + LG_LP_S - 1) / LG_LP_S;
    const int ck = a.dimp >> 3, cr = a.rotp >> 3, cv = a.vdp >> 3;
    auto load_tile = [&](int tile, int buf) {
        bf16 *dk = sK + (size_t)buf * LG_LP_S * lq, *dv = sV + (size_t)buf * LG_LP_S * lv;
        const int k0 = tile * LG_LP_S, per = ck + cr + cv;
        for (int u = tid; u < LG_LP_S * per; u += LG_LP_THREADS) {
            const int r = u / per, c = u % per;
            const size_t key = k0 + r;
            bf16 *dst = c < ck + cr ? dk + (size_t)r * lq + c * 8 : dv + (size_t)r * lv + (c - ck - cr) * 8;
            if (k0 + r >= n_keys) { *(uint4 *)dst = make_uint4(0, 0, 0, 0); continue; }
            const bf16 *src = c < ck ? a.ex + key * a.ldx + h * a.dimp + c * 8
                            : c < ck + cr ? a.cache + key * a.ldc + a.rot_at + (c - ck) * 8
                            : a.ex + key * a.ldx + a.H * a.dimp + h * a.vdp + (c - ck - cr) * 8;
            cp_async16(dst, src);
        }
        cp_async_commit();
    };
    load_tile(0, 0);
    for (int u = tid; u < LG_LP_Q * (dq >> 3); u += LG_LP_THREADS) {
        const int r = u / (dq >> 3), c = u % (dq >> 3) * 8, tok = qb + r;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (tok < a.n) {
            v = *(const uint4 *)(a.q + (size_t)tok * a.ldq + (size_t)h * dq + c);
            if (c >= a.dimp) {
                uint32_t *w = (uint32_t *)&v;
                const float2 *tb = a.tab + (size_t)tok * (a.rot_dims >> 1);
                #pragma unroll
                for (int i = 0; i < 4; i++) {
                    const int pair = ((c - a.dimp) >> 1) + i;
                    if (2 * pair >= a.rot_dims) break;
                    const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *)&w[i]), cs = tb[pair];
                    w[i] = pack_bf16(x.x * cs.x - x.y * cs.y, x.y * cs.x + x.x * cs.y);
                }
            }
        }
        *(uint4 *)(sQ + (size_t)r * lq + c) = v;
    }
    float acc[NV][4];
    #pragma unroll
    for (int n = 0; n < NV; n++)
        #pragma unroll
        for (int i = 0; i < 4; i++) acc[n][i] = 0.0f;
    const float sc = a.scale * LG_LOG2E, sink = a.sink[h] * LG_LOG2E;
    float m0 = sink, m1 = sink, l0 = t == 0 ? 1.0f : 0.0f, l1 = l0;              // (a row's sum is spread over four lanes)
    const int wq = qb + warp * 16, q_lo = pos + wq + g, q_hi = q_lo + 8;          // this lane's two query positions
    const int warp_keys = pos + wq + 16;                                          // keys past these are masked for the whole warp
    int buf = 0;
    for (int tile = 0; tile < n_tiles; tile++, buf ^= 1) {
        __syncthreads();                               // everyone has left the buffer the next copy overwrites (first pass: Q is stored)
        if (tile + 1 < n_tiles) { load_tile(tile + 1, buf ^ 1); cp_async_wait<1>(); } else cp_async_wait<0>();
        __syncthreads();
        const int k0 = tile * LG_LP_S;
        if (k0 >= warp_keys) continue;                 // (the barriers above are reached by every warp in every pass)
        const bf16 *K = sK + (size_t)buf * LG_LP_S * lq, *V = sV + (size_t)buf * LG_LP_S * lv;
        float s[8][4];
        #pragma unroll
        for (int n = 0; n < 8; n++)
            #pragma unroll
            for (int i = 0; i < 4; i++) s[n][i] = 0.0f;
        const bf16 *qp = sQ + (size_t)(warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * lq + ((lane >> 4) & 1) * 8;
        const bf16 *kp = K + (size_t)((lane & 7) + ((lane >> 4) & 1) * 8) * lq + ((lane >> 3) & 1) * 8;
        #pragma unroll 4
        for (int kk = 0; kk < dq >> 4; kk++) {
            uint32_t q4[4];
            ldsm_x4(q4, qp + kk * 16);
            #pragma unroll
            for (int n = 0; n < 4; n++) {
                uint32_t b[4];
                ldsm_x4(b, kp + (size_t)n * 16 * lq + kk * 16);
                mma_bf16(s[2 * n], q4[0], q4[1], q4[2], q4[3], b[0], b[1]);
                mma_bf16(s[2 * n + 1], q4[0], q4[1], q4[2], q4[3], b[2], b[3]);
            }
        }
        const bool edge = k0 + LG_LP_S > pos + wq + 1;
        float mx0 = -INFINITY, mx1 = -INFINITY;
        #pragma unroll
        for (int n = 0; n < 8; n++)
            #pragma unroll
            for (int i = 0; i < 4; i++) {
                const int key = k0 + n * 8 + 2 * t + (i & 1);
                s[n][i] = edge && key > (i < 2 ? q_lo : q_hi) ? -INFINITY : s[n][i] * sc;
                if (i < 2) mx0 = fmaxf(mx0, s[n][i]); else mx1 = fmaxf(mx1, s[n][i]);
            }
        #pragma unroll
        for (int o = 1; o <= 2; o <<= 1) { mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, o)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, o)); }
        const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1), a0 = exp2f(m0 - n0), a1 = exp2f(m1 - n1);
        m0 = n0; m1 = n1; l0 *= a0; l1 *= a1;
        #pragma unroll
        for (int n = 0; n < 8; n++) {
            s[n][0] = exp2f(s[n][0] - n0); s[n][1] = exp2f(s[n][1] - n0); s[n][2] = exp2f(s[n][2] - n1); s[n][3] = exp2f(s[n][3] - n1);
            l0 += s[n][0] + s[n][1]; l1 += s[n][2] + s[n][3];
        }
        #pragma unroll
        for (int n = 0; n < NV; n++) { acc[n][0] *= a0; acc[n][1] *= a0; acc[n][2] *= a1; acc[n][3] *= a1; }
        const bf16 *vp = V + (size_t)((lane & 7) + ((lane >> 3) & 1) * 8) * lv + ((lane >> 4) & 1) * 8;
        #pragma unroll
        for (int j = 0; j < 4; j++) {
            uint32_t ph[4], pl[4];
            split_bf16(s[2 * j][0], s[2 * j][1], ph[0], pl[0]); split_bf16(s[2 * j][2], s[2 * j][3], ph[1], pl[1]);
            split_bf16(s[2 * j + 1][0], s[2 * j + 1][1], ph[2], pl[2]); split_bf16(s[2 * j + 1][2], s[2 * j + 1][3], ph[3], pl[3]);
            #pragma unroll
            for (int n = 0; n < NV; n += 2) {
                if (n * 8 >= a.vdp) break;
                uint32_t v[4];
                ldsm_x4_t(v, vp + (size_t)j * 16 * lv + n * 8);
                mma_bf16(acc[n], ph[0], ph[1], ph[2], ph[3], v[0], v[1]);
                mma_bf16(acc[n], pl[0], pl[1], pl[2], pl[3], v[0], v[1]);
                mma_bf16(acc[n + 1], ph[0], ph[1], ph[2], ph[3], v[2], v[3]);
                mma_bf16(acc[n + 1], pl[0], pl[1], pl[2], pl[3], v[2], v[3]);
            }
        }
    }
    #pragma unroll
    for (int o = 1; o <= 2; o <<= 1) { l0 += __shfl_xor_sync(0xffffffffu, l0, o); l1 += __shfl_xor_sync(0xffffffffu, l1, o); }
    const float i0 = 1.0f / l0, i1 = 1.0f / l1;
    #pragma unroll
    for (int n = 0; n < NV; n++) {
        const int col = n * 8 + 2 * t;
        if (n * 8 >= a.vdp) break;
        #pragma unroll
        for (int r = 0; r < 2; r++) {
            const int tok = wq + g + 8 * r;
            if (tok >= a.n) continue;
            const float2 gt = *(const float2 *)(a.gate + (size_t)tok * a.ldg + h * a.vdp + col);
            const float iv = r ? i1 : i0;
            *(uint32_t *)(a.out + (size_t)tok * a.ldo + h * a.vdp + col) =
                pack_bf16(acc[n][2 * r] * iv * sigmoid_f(gt.x), acc[n][2 * r + 1] * iv * sigmoid_f(gt.y));
        }
    }
}
