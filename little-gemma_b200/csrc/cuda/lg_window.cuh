// lg_window.cuh -- grouped attention over cached key / value rows, within a sliding window, with one or two softmax maps per head.
//
// A cache row holds [ keys: G x MAPS x dimp | values: G x vdp ]; position p lies in row p % seq (seq a multiple of 64, so a tile of 64
// positions on absolute boundaries never straddles the wrap).  Query head h reads group h / (H / G).  Position i sees j with
// 0 <= i - j < window (window 0: every earlier position).  With two maps (differential attention) each has a softmax of its own over the
// same values, and the head's output is  o = a1 - lambda a2,  o / sqrt(mean(o^2) + eps) * out_mult;  with one map it is a1.
//
//  * lg_win_attn_rows_kernel: one (token, head) per CTA in f32 arithmetic, for 32-bit models and sizes the others do not hold;
//  * lg_win_dec_attn_kernel + lg_win_merge_kernel: decode / verify, split over key tiles;
//  * lg_win_pf_attn_kernel: prompt blocks, on tcgen05.
#pragma once
#include "lg_seq.cuh"
#include "lg_ssd.cuh"               // MN-major operands

struct LgWinArgs {
    const void *q; int ldq;                      // [token][H][MAPS][dimp]
    const void *cache; int ldc, v_off, seq;
    int H, G, dimp, vd, vdp, window;
    float scale, lambda, out_mult, eps;
    const int *pos; int n;                       // position of token 0; tokens
    void *out; int ldo;                          // [token][H][vdp]
    float *part; float2 *part_ml;                // decode: [C][row][vdp], [C][row]; row = (token H + h) MAPS + map
    int *err;
};
// first position that position p sees
__host__ __device__ __forceinline__ int lg_win_first(int p, int window) { return window > 0 && p >= window ? p - window + 1 : 0; }

// ---------------------------------------------------------------------------------------------
// one (token, head) per CTA, f32 arithmetic
// ---------------------------------------------------------------------------------------------
template <typename T, int MAPS>
__global__ void __launch_bounds__(128) lg_win_attn_rows_kernel(LgWinArgs a) {
    extern __shared__ __align__(16) unsigned char win_smem[];
    constexpr int S = 128;
    float *sq = (float *)win_smem, *acc = sq + MAPS * a.dimp, *sp = acc + MAPS * a.vdp;
    __shared__ float red[32];
    pdl_launch(); pdl_wait();
    const int h = blockIdx.x, tok = blockIdx.y, g = h / (a.H / a.G), lane = threadIdx.x & 31, warp = threadIdx.x >> 5, p = *a.pos + tok;
    const T *q = (const T *)a.q + (size_t)tok * a.ldq + (size_t)h * MAPS * a.dimp, *cache = (const T *)a.cache;
    for (int i = threadIdx.x; i < MAPS * a.dimp; i += blockDim.x) sq[i] = from_elem(q[i]);
    for (int i = threadIdx.x; i < MAPS * a.vdp; i += blockDim.x) acc[i] = 0.0f;
    __syncthreads();
    float m[MAPS], l[MAPS];
    #pragma unroll
    for (int x = 0; x < MAPS; x++) { m[x] = -INFINITY; l[x] = 0.0f; }
    const float sc = a.scale * LG_LOG2E;
    for (int k0 = lg_win_first(p, a.window); k0 <= p; k0 += S) {
        const int nk = min(S, p + 1 - k0);
        for (int k = warp; k < nk; k += 4) {
            const T *c = cache + (size_t)((k0 + k) % a.seq) * a.ldc + (size_t)g * MAPS * a.dimp;
            #pragma unroll
            for (int x = 0; x < MAPS; x++) {
                float d = 0.0f;
                for (int i = lane; i < a.dimp; i += 32) d = fmaf(sq[x * a.dimp + i], from_elem(c[x * a.dimp + i]), d);
                d = warp_sum(d);
                if (lane == 0) sp[x * S + k] = d * sc;
            }
        }
        __syncthreads();
        float alpha[MAPS];
        #pragma unroll
        for (int x = 0; x < MAPS; x++) {
            const float s = threadIdx.x < nk ? sp[x * S + threadIdx.x] : -INFINITY;
            float mx = warp_max(s);
            if (lane == 0) red[warp] = mx;
            __syncthreads();
            mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
            const float m_new = fmaxf(m[x], mx), w = threadIdx.x < nk ? exp2f(s - m_new) : 0.0f;
            alpha[x] = exp2f(m[x] - m_new);          // the first tile has a visible key, so m_new is finite
            const float tot = block_sum(w, red);     // (its barriers order the reads of red and sp above before the writes below)
            if (threadIdx.x < nk) sp[x * S + threadIdx.x] = w;
            __syncthreads();
            l[x] = l[x] * alpha[x] + tot; m[x] = m_new;
        }
        for (int i = threadIdx.x; i < a.vdp; i += blockDim.x) {
            float o[MAPS];
            #pragma unroll
            for (int x = 0; x < MAPS; x++) o[x] = acc[x * a.vdp + i] * alpha[x];
            for (int k = 0; k < nk; k++) {
                const float v = from_elem(cache[(size_t)((k0 + k) % a.seq) * a.ldc + a.v_off + g * a.vdp + i]);
                #pragma unroll
                for (int x = 0; x < MAPS; x++) o[x] = fmaf(sp[x * S + k], v, o[x]);
            }
            #pragma unroll
            for (int x = 0; x < MAPS; x++) acc[x * a.vdp + i] = o[x];
        }
        __syncthreads();
    }
    T *out = (T *)a.out + (size_t)tok * a.ldo + (size_t)h * a.vdp;
    if (MAPS == 1) {
        for (int i = threadIdx.x; i < a.vdp; i += blockDim.x) to_elem(acc[i] / l[0], out[i]);
        return;
    }
    const float c1 = 1.0f / l[0], c2 = a.lambda / l[MAPS - 1];
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.vdp; i += blockDim.x) {
        const float o = acc[i] * c1 - acc[(MAPS - 1) * a.vdp + i] * c2;
        acc[i] = o;
        ss = fmaf(o, o, ss);
    }
    const float f = a.out_mult / sqrtf(block_sum(ss, red) / (float)a.vd + a.eps);
    for (int i = threadIdx.x; i < a.vdp; i += blockDim.x) to_elem(acc[i] * f, out[i]);
}

// ---------------------------------------------------------------------------------------------
// decode / verify: split over key tiles
// ---------------------------------------------------------------------------------------------
// CTA (x, g, z): group g, query rows [16 z, 16 z + 16) of the block's (token, head of the group) rows, both maps; key tiles t of 64
// positions with t % C == x (C = gridDim.x comes from the cache length, the window and G alone), online softmax, one partial
// (max, sum, value row) per row and map.  Tiles arrive by tiled TMA copies; the first one is requested before the dependency wait unless it
// holds rows of this very step.  A row's arithmetic depends neither on the rows beside it nor on the width of the block.
#define LG_WD_S 64
#define LG_WD_THREADS 256
__host__ __device__ constexpr size_t lg_win_dec_smem(int maps, int dimp, int vdp) {
    return 1024 + (size_t)2 * (maps * lg_ssd_blocks(dimp) + lg_ssd_blocks(vdp)) * LG_WD_S * 128
         + (size_t)maps * 16 * ((dimp + 8) * 2 + 2 * (LG_WD_S + 8) * 2 + (LG_WD_S + 4) * 4 + 3 * 4) + 32;
}
template <int MAPS, int NACC>
__global__ void __launch_bounds__(LG_WD_THREADS, 1) lg_win_dec_attn_kernel(const __grid_constant__ CUtensorMap tmc, LgWinArgs a) {
    extern __shared__ __align__(16) unsigned char win_smem[];
    constexpr int S = LG_WD_S, LP = S + 8, LS = S + 4, R = MAPS * 16, TILE = S * 128;
    const int lq = a.dimp + 8, kb = lg_ssd_blocks(a.dimp), vb = lg_ssd_blocks(a.vdp), nblk = MAPS * kb + vb;
    unsigned char *sK = (unsigned char *)(((uintptr_t)win_smem + 1023) & ~(uintptr_t)1023);
    bf16 *sQ = (bf16 *)(sK + 2 * nblk * TILE), *sPh = sQ + R * lq, *sPl = sPh + R * LP;
    float *sS = (float *)(sPl + R * LP), *sM = sS + R * LS, *sL = sM + R, *sA = sL + R;
    uint64_t *full = (uint64_t *)(((uintptr_t)(sA + R) + 7) & ~(uintptr_t)7);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t4 = lane & 3;
    const int C = gridDim.x, g = blockIdx.y, hpg = a.H / a.G, rows = a.n * hpg, row0 = blockIdx.z * 16;
    pdl_launch();
    const int pos = *a.pos;                                        // the position and every row below it come from earlier forwards
    const int last_row = min(row0 + 16, rows) - 1, tok_lo = row0 / hpg, tok_hi = last_row / hpg;
    const int t_lo = lg_win_first(pos + tok_lo, a.window) / S, t_hi = (pos + tok_hi) / S;
    int tile = t_lo + ((int)blockIdx.x - t_lo % C + C) % C;        // the first of this CTA's tiles that the rows see
    if (tile > t_hi) return;
    auto load_tile = [&](int t, int buf) {                         // thread 0
        unsigned char *d = sK + buf * nblk * TILE;
        const int row = (int)(((long long)t * S) % a.seq);
        mbar_expect_tx(full + buf, nblk * TILE);
        for (int m = 0; m < MAPS; m++)
            for (int c = 0; c < kb; c++) tma_load_2d(d + (m * kb + c) * TILE, &tmc, (g * MAPS + m) * a.dimp + c * 64, row, full + buf);
        for (int c = 0; c < vb; c++) tma_load_2d(d + (MAPS * kb + c) * TILE, &tmc, a.v_off + g * a.vdp + c * 64, row, full + buf);
    };
    const bool early = (tile + 1) * S <= pos;
    if (tid == 0) {
        mbar_init(full, 1); mbar_init(full + 1, 1);
        if (early) load_tile(tile, 0);
    }
    if (tid < R) { sM[tid] = -INFINITY; sL[tid] = 0.0f; }
    pdl_wait();
    if (tid == 0 && !early) load_tile(tile, 0);
    const int cpr = a.dimp >> 3;
    for (int r = warp; r < R; r += LG_WD_THREADS / 32) {
        const int rr = row0 + (r & 15), m = r >> 4;
        const bf16 *src = (const bf16 *)a.q + (size_t)(rr / hpg) * a.ldq + (size_t)((g * hpg + rr % hpg) * MAPS + m) * a.dimp;
        for (int c = lane; c < cpr; c += 32) *(uint4 *)(sQ + (size_t)r * lq + c * 8) = rr < rows ? *(const uint4 *)(src + c * 8) : make_uint4(0, 0, 0, 0);
    }
    constexpr int WPM = 8 / MAPS;                                  // warps per map in the value product
    const int om = warp / WPM, col0 = (warp % WPM) * NACC * 8;
    float acc[NACC][4];
    #pragma unroll
    for (int n = 0; n < NACC; n++)
        #pragma unroll
        for (int i = 0; i < 4; i++) acc[n][i] = 0.0f;
    const int sm = warp >> 2, kg = warp & 3;                       // scores: map, group of 16 keys
    const float sc = a.scale * LG_LOG2E;
    const int qr = (lane & 7) + ((lane >> 3) & 1) * 8, qc = ((lane >> 4) & 1) * 8;               // this lane's row / column of a 16 x 16 A block
    const int kr = kg * 16 + (lane & 7) + ((lane >> 4) & 1) * 8, kc = (lane >> 3) & 1;           // key row and 8-column half of a B block
    const int x7 = lane & 7;
    __syncthreads();
    uint32_t ph = 0;
    int buf = 0;
    bool ok = true;
    for (; tile <= t_hi; tile += C, buf ^= 1) {
        if (tid == 0 && tile + C <= t_hi) load_tile(tile + C, buf ^ 1);
        if (ok && !mbar_wait(full + buf, (ph >> buf) & 1)) { ok = false; if (lane == 0) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT); }
        ph ^= 1u << buf;
        const unsigned char *K = sK + buf * nblk * TILE;
        if (sm < MAPS) {
            float s[2][4] = {};
            const unsigned char *kp = K + sm * kb * TILE + kr * 128;
            const bf16 *qp = sQ + (size_t)(sm * 16 + qr) * lq + qc;
            #pragma unroll 4
            for (int kk = 0; kk < a.dimp >> 4; kk++) {
                uint32_t b[4], q4[4];
                ldsm_x4(b, kp + (kk >> 2) * TILE + ((((kk & 3) * 2 + kc) ^ x7) << 4));
                ldsm_x4(q4, qp + kk * 16);
                mma_bf16(s[0], q4[0], q4[1], q4[2], q4[3], b[0], b[1]);
                mma_bf16(s[1], q4[0], q4[1], q4[2], q4[3], b[2], b[3]);
            }
            #pragma unroll
            for (int n = 0; n < 2; n++) {
                float *d = sS + (size_t)(sm * 16 + gq) * LS + kg * 16 + n * 8 + 2 * t4;
                *(float2 *)d = make_float2(s[n][0], s[n][1]);
                *(float2 *)(d + 8 * LS) = make_float2(s[n][2], s[n][3]);
            }
        }
        __syncthreads();
        #pragma unroll
        for (int rr = 0; rr < R / 8; rr++) {           // softmax: a warp per row, two keys per lane
            const int r = warp * (R / 8) + rr, row = row0 + (r & 15);
            const float2 s0 = *(const float2 *)(sS + (size_t)r * LS + 2 * lane);
            const int key = tile * S + 2 * lane, seen = row < rows ? pos + row / hpg : -1, lo = lg_win_first(seen, a.window);
            const float v0 = key <= seen && key >= lo ? s0.x * sc : -INFINITY, v1 = key + 1 <= seen && key + 1 >= lo ? s0.y * sc : -INFINITY;
            const float m_old = sM[r], m_new = fmaxf(m_old, warp_max(fmaxf(v0, v1)));
            const float p0 = m_new == -INFINITY ? 0.0f : exp2f(v0 - m_new), p1 = m_new == -INFINITY ? 0.0f : exp2f(v1 - m_new);
            const float sum = warp_sum(p0 + p1);
            uint32_t hi, lw;
            split_bf16(p0, p1, hi, lw);
            *(uint32_t *)(sPh + r * LP + 2 * lane) = hi;
            *(uint32_t *)(sPl + r * LP + 2 * lane) = lw;
            if (lane == 0) {
                const float al = m_old == -INFINITY ? 0.0f : exp2f(m_old - m_new);
                sA[r] = al; sM[r] = m_new; sL[r] = sL[r] * al + sum;
            }
        }
        __syncthreads();
        if (col0 < a.vdp) {
            const float a0 = sA[om * 16 + gq], a1 = sA[om * 16 + gq + 8];
            #pragma unroll
            for (int n = 0; n < NACC; n++) { acc[n][0] *= a0; acc[n][1] *= a0; acc[n][2] *= a1; acc[n][3] *= a1; }
            const unsigned char *vp = K + MAPS * kb * TILE + qr * 128;
            const int po = (om * 16 + qr) * LP + qc;
            #pragma unroll
            for (int k16 = 0; k16 < S / 16; k16++) {
                uint32_t p4h[4], p4l[4];
                ldsm_x4(p4h, sPh + po + k16 * 16);
                ldsm_x4(p4l, sPl + po + k16 * 16);
                #pragma unroll
                for (int n = 0; n < NACC; n += 2) {
                    const int c8 = (col0 >> 3) + n;                      // 8-column group
                    if (c8 * 8 >= a.vdp) break;
                    uint32_t v[4];
                    ldsm_x4_t(v, vp + k16 * 16 * 128 + (c8 >> 3) * TILE + ((((c8 & 7) + (qc >> 3)) ^ x7) << 4));
                    mma_bf16(acc[n], p4h[0], p4h[1], p4h[2], p4h[3], v[0], v[1]);
                    mma_bf16(acc[n + 1], p4h[0], p4h[1], p4h[2], p4h[3], v[2], v[3]);
                    mma_bf16(acc[n], p4l[0], p4l[1], p4l[2], p4l[3], v[0], v[1]);
                    mma_bf16(acc[n + 1], p4l[0], p4l[1], p4l[2], p4l[3], v[2], v[3]);
                }
            }
        }
        __syncthreads();                               // the tile's buffer is free for the copy after next
    }
    const size_t all = (size_t)a.n * a.H * MAPS;
    auto out_row = [&](int r, int m) { return ((size_t)(r / hpg) * a.H + g * hpg + r % hpg) * MAPS + m; };
    #pragma unroll
    for (int n = 0; n < NACC; n++) {
        const int col = col0 + n * 8 + 2 * t4;
        if (col >= a.vdp) continue;
        #pragma unroll
        for (int i = 0; i < 2; i++) {
            const int r = row0 + gq + 8 * i;
            if (r < rows) *(float2 *)(a.part + ((size_t)blockIdx.x * all + out_row(r, om)) * a.vdp + col) = make_float2(acc[n][2 * i], acc[n][2 * i + 1]);
        }
    }
    if (tid < R && row0 + (tid & 15) < rows) a.part_ml[(size_t)blockIdx.x * all + out_row(row0 + (tid & 15), tid >> 4)] = make_float2(sM[tid], sL[tid]);
}

// Merge of the partials and the combination of the maps: bf16 rows.  One CTA per token and head; group q of its threads takes splits q,
// q + GROUPS, ... counted from the split of the row's first visible tile.
#define LG_WM_GROUPS 4
#define LG_WM_THREADS 512
#define LG_WM_MAXC 160
template <int MAPS>
__global__ void __launch_bounds__(LG_WM_THREADS) lg_win_merge_kernel(LgWinArgs a, int C) {
    __shared__ __align__(16) float sum[LG_WM_GROUPS][MAPS * 256];
    __shared__ float w[MAPS][LG_WM_MAXC], s_inv[MAPS], red[32];
    pdl_launch();
    const int tok = blockIdx.x / a.H, h = blockIdx.x % a.H, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int p = *a.pos + tok, t_lo = lg_win_first(p, a.window) / LG_WD_S, n = min(C, p / LG_WD_S - t_lo + 1);
    constexpr int TPG = LG_WM_THREADS / LG_WM_GROUPS;
    const int grp = tid / TPG, c = (tid % TPG) * 4, cols = MAPS * a.vdp, m = c < a.vdp ? 0 : MAPS - 1;
    const size_t all = (size_t)a.n * a.H * MAPS, row = (size_t)blockIdx.x * MAPS;
    pdl_wait();
    if (warp < MAPS) {
        float mx = -INFINITY, l = 0.0f;
        for (int i = lane; i < n; i += 32) mx = fmaxf(mx, a.part_ml[(size_t)((t_lo + i) % C) * all + row + warp].x);
        mx = warp_max(mx);
        for (int i = lane; i < n; i += 32) {
            const float2 ml = a.part_ml[(size_t)((t_lo + i) % C) * all + row + warp];
            const float e = ml.x == -INFINITY ? 0.0f : exp2f(ml.x - mx);
            w[warp][i] = e;
            l = fmaf(ml.y, e, l);
        }
        l = warp_sum(l);
        if (lane == 0) s_inv[warp] = 1.0f / l;
    }
    __syncthreads();
    if (c < cols) {
        float4 o = make_float4(0, 0, 0, 0);
        #pragma unroll 4
        for (int i = grp; i < n; i += LG_WM_GROUPS) {
            const float4 x = *(const float4 *)(a.part + ((size_t)((t_lo + i) % C) * all + row) * a.vdp + c);         // the maps' rows are neighbours
            const float wi = w[m][i];
            o.x = fmaf(wi, x.x, o.x); o.y = fmaf(wi, x.y, o.y); o.z = fmaf(wi, x.z, o.z); o.w = fmaf(wi, x.w, o.w);
        }
        *(float4 *)&sum[grp][c] = o;
    }
    __syncthreads();
    float o = 0.0f;
    if (tid < a.vdp) {
        #pragma unroll
        for (int x = 0; x < MAPS; x++) {
            float s = 0.0f;
            #pragma unroll
            for (int q = 0; q < LG_WM_GROUPS; q++) s += sum[q][x * a.vdp + tid];
            o = x == 0 ? s * s_inv[0] : o - a.lambda * (s * s_inv[x]);
        }
    }
    if (MAPS > 1) o *= a.out_mult / sqrtf(block_sum(o * o, red) / (float)a.vd + a.eps);
    if (tid < a.vdp) ((bf16 *)a.out)[(size_t)tok * a.ldo + (size_t)h * a.vdp + tid] = __float2bfloat16_rn(o);
}

// ---------------------------------------------------------------------------------------------
// prompt blocks: on tcgen05
// ---------------------------------------------------------------------------------------------
// CTA = one head (all its maps) x 128 query rows (the TMEM lanes), key tiles of 64 from the first one any row sees.  Warps:
//   0 .. 4 MAPS - 1   map w / 4, one query row per thread: online softmax in f32, the weights back over the scores in tensor memory as bf16
//                     high + low parts; the output is rescaled only when a row's maximum has grown by more than 2^LG_LP_SLACK;
//   then one thread each:  Q and key tiles;  products;  value tiles (keys and values in two stages).
// Scores of two tiles may be finished before the first one's weights are used, so every buffer has barriers of its own, for its weights and
// for the product with them: of one barrier for both, a parity could stand for the phase before or after the one that is waited for.  Per map tensor memory holds two score buffers of 64 columns and the output; values are an MN-major operand, as they lie in the cache.
// At the end both maps' rows sit in the same lanes: warps w and w + 4 share a row's columns, combine and norm them.
#define LG_WP_Q 128
#define LG_WP_S 64
#define LG_WP_STAGES 2
__host__ __device__ constexpr size_t lg_win_pf_smem(int maps, int dimp, int vdp) {
    return 1024 + (size_t)maps * lg_ssd_blocks(dimp) * (LG_WP_Q + LG_WP_STAGES * LG_WP_S) * 128 + (size_t)LG_WP_STAGES * lg_ssd_blocks(vdp) * LG_WP_S * 128 + 256;
}
template <int MAPS> constexpr int lg_win_pf_threads() { return MAPS * 128 + 96; }
template <int MAPS>
__global__ void __launch_bounds__(MAPS * 128 + 96, 1)
lg_win_pf_attn_kernel(const __grid_constant__ CUtensorMap tmq, const __grid_constant__ CUtensorMap tmc, LgWinArgs a) {
    extern __shared__ __align__(16) unsigned char win_smem[];
    __shared__ float s_l[MAPS][LG_WP_Q], s_ss[MAPS][LG_WP_Q];
    constexpr int ST = LG_WP_STAGES, Q_BYTES = LG_WP_Q * 128, T_BYTES = LG_WP_S * 128, ROWW = 4 * MAPS;
    const int kb = lg_ssd_blocks(a.dimp), vb = lg_ssd_blocks(a.vdp), nb = MAPS * kb, vo = (a.vdp + 31) & ~31;
    unsigned char *sQ = (unsigned char *)(((uintptr_t)win_smem + 1023) & ~(uintptr_t)1023), *sK = sQ + nb * Q_BYTES, *sV = sK + ST * nb * T_BYTES;
    uint64_t *qfull = (uint64_t *)(sV + ST * vb * T_BYTES), *kfull = qfull + 1, *kempty = kfull + ST, *vfull = kempty + ST, *vempty = vfull + ST,
             *sfull = vempty + ST /* [map][2] */, *pready = sfull + 2 * MAPS /* [map][2] */, *odone = pready + 2 * MAPS /* [map][2] */;
    uint32_t *tmem_slot = (uint32_t *)(odone + 2 * MAPS);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y, g = h / (a.H / a.G), qb = (gridDim.x - 1 - blockIdx.x) * LG_WP_Q;       // longest rows first
    const uint32_t tcols = lg_tmem_cols(MAPS * (2 * LG_WP_S + vo));
    if (threadIdx.x == 0) {
        mbar_init(qfull, 1);
        for (int i = 0; i < ST; i++) { mbar_init(kfull + i, 1); mbar_init(kempty + i, 1); mbar_init(vfull + i, 1); mbar_init(vempty + i, 1); }
        for (int i = 0; i < MAPS; i++) { mbar_init(sfull + 2 * i, 1); mbar_init(sfull + 2 * i + 1, 1); mbar_init(pready + 2 * i, 128); mbar_init(pready + 2 * i + 1, 128); mbar_init(odone + 2 * i, 1); mbar_init(odone + 2 * i + 1, 1); }
    }
    if (warp == ROWW + 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(smem_u32(tmem_slot)), "r"(tcols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot, tO = tmem + MAPS * 2 * LG_WP_S;
    pdl_launch();                        // only now: a dependant must not take tensor memory a CTA of this grid still waits for
    pdl_wait();
    const int pos = *a.pos, q_last = pos + min(qb + LG_WP_Q, a.n) - 1;
    const int t0 = lg_win_first(pos + qb, a.window) / LG_WP_S, n_tiles = q_last / LG_WP_S - t0 + 1;
    auto cache_row = [&](int i) { return (int)(((long long)(t0 + i) * LG_WP_S) % a.seq); };

    if (warp == ROWW) {
        if (lane == 0) {
            mbar_expect_tx(qfull, nb * Q_BYTES);
            for (int m = 0; m < MAPS; m++)
                for (int c = 0; c < kb; c++) tma_load_2d(sQ + (m * kb + c) * Q_BYTES, &tmq, (h * MAPS + m) * a.dimp + c * 64, qb, qfull);
            int i = 0;
            for (; i < n_tiles; i++) {
                const int s = i % ST;
                if (i >= ST && !mbar_wait(kempty + s, (i / ST - 1) & 1)) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 2048); break; }
                mbar_expect_tx(kfull + s, nb * T_BYTES);
                for (int m = 0; m < MAPS; m++)
                    for (int c = 0; c < kb; c++) tma_load_2d(sK + (s * nb + m * kb + c) * T_BYTES, &tmc, (g * MAPS + m) * a.dimp + c * 64, cache_row(i), kfull + s);
            }
            if (i < n_tiles) {           // own copies in flight land before the CTA ends
                mbar_wait(qfull, 0);
                for (int j = max(0, i - ST); j < i; j++) mbar_wait(kfull + j % ST, (j / ST) & 1);
            }
        }
    } else if (warp == ROWW + 2) {
        if (lane == 0) {
            int i = 0;
            for (; i < n_tiles; i++) {
                const int s = i % ST;
                if (i >= ST && !mbar_wait(vempty + s, (i / ST - 1) & 1)) { atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 4096); break; }
                mbar_expect_tx(vfull + s, vb * T_BYTES);
                for (int c = 0; c < vb; c++) tma_load_2d(sV + (s * vb + c) * T_BYTES, &tmc, a.v_off + g * a.vdp + c * 64, cache_row(i), vfull + s);
            }
            if (i < n_tiles) for (int j = max(0, i - ST); j < i; j++) mbar_wait(vfull + j % ST, (j / ST) & 1);
        }
    } else if (warp == ROWW + 1) {
        if (lane == 0) {
            // f32 accumulator, bf16 x bf16; N = keys of a tile / value columns
            const uint32_t fmt = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(LG_WP_Q >> 4) << 24);
            const uint32_t idS = fmt | ((uint32_t)(LG_WP_S >> 3) << 17), idO = fmt | ((uint32_t)(a.vdp >> 3) << 17) | LG_UMMA_B_MN;
            const int steps = a.dimp >> 4;
            bool ok = mbar_wait(qfull, 0);
            auto scores = [&](int i) {
                const int s = i % ST;
                if (!mbar_wait(kfull + s, (i / ST) & 1)) return false;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                #pragma unroll
                for (int m = 0; m < MAPS; m++) {
                    const uint64_t qd = umma_desc_k128(smem_u32(sQ + m * kb * Q_BYTES)), kd = umma_desc_k128(smem_u32(sK + (s * nb + m * kb) * T_BYTES));
                    for (int j = 0; j < steps; j++)
                        umma_f16(tmem + (2 * m + (i & 1)) * LG_WP_S, qd + (j >> 2) * (Q_BYTES >> 4) + 2 * (j & 3), kd + (j >> 2) * (T_BYTES >> 4) + 2 * (j & 3), idS, j ? 1u : 0u);
                    umma_commit(sfull + 2 * m + (i & 1));
                }
                umma_commit(kempty + s);
                return true;
            };
            ok = ok && scores(0);
            for (int i = 0; i < n_tiles && ok; i++) {
                if (i + 1 < n_tiles) ok = scores(i + 1);
                const int s = i % ST;
                ok = ok && mbar_wait(vfull + s, (i / ST) & 1);
                #pragma unroll
                for (int m = 0; m < MAPS; m++) {
                    ok = ok && mbar_wait(pready + 2 * m + (i & 1), (i >> 1) & 1);
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint64_t vd = umma_desc_mn128(smem_u32(sV + s * vb * T_BYTES), T_BYTES);
                    const uint32_t tP = tmem + (2 * m + (i & 1)) * LG_WP_S;
                    #pragma unroll
                    for (int j = 0; j < 4; j++) umma_f16_ta(tO + m * vo, tP + 8 * j, vd + 128 * j, idO, (i | j) ? 1u : 0u);
                    #pragma unroll
                    for (int j = 0; j < 4; j++) umma_f16_ta(tO + m * vo, tP + 32 + 8 * j, vd + 128 * j, idO, 1u);
                    umma_commit(odone + 2 * m + (i & 1));
                }
                umma_commit(vempty + s);
            }
            if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 8192);
        }
    } else {
        const int map = warp >> 2, row = threadIdx.x & 127, tok = qb + row, q_pos = pos + tok, q_lo = lg_win_first(q_pos, a.window);
        const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
        const float sc = a.scale * LG_LOG2E;
        // tiles in [whole_lo, whole_hi) are seen whole by every row of the warp
        const int w_first = pos + qb + (warp & 3) * 32;
        const int whole_hi = (w_first + 1) / LG_WP_S, whole_lo = (lg_win_first(w_first + 31, a.window) + LG_WP_S - 1) / LG_WP_S;
        float m = -1e30f, l = 0.0f;
        bool ok = true;
        for (int i = 0; i < n_tiles; i++) {
            ok = __all_sync(0xffffffffu, mbar_wait(sfull + 2 * map + (i & 1), (i >> 1) & 1));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t tS = tmem + lanes + (2 * map + (i & 1)) * LG_WP_S;
            uint32_t s0[32], s1[32];
            __syncwarp();
            tmem_ld32(tS, s0);
            tmem_ld32(tS + 32, s1);
            const int tile = t0 + i;
            float mx = -INFINITY;
            if (tile >= whole_hi || tile < whole_lo) {
                #pragma unroll
                for (int j = 0; j < 32; j++) {
                    const int key = tile * LG_WP_S + j;
                    if (key > q_pos || key < q_lo) s0[j] = 0xff800000u;
                    if (key + 32 > q_pos || key + 32 < q_lo) s1[j] = 0xff800000u;
                }
            }
            #pragma unroll
            for (int j = 0; j < 32; j++) mx = fmaxf(mx, fmaxf(__uint_as_float(s0[j]), __uint_as_float(s1[j])));
            const float mt = mx * sc;                          // a row's scores are scaled in the exponent: exp2(s * sc - m)
            const bool grow = i == 0 || mt > m + LG_LP_SLACK;
            if (__any_sync(0xffffffffu, grow)) {
                const float m_new = fmaxf(m, mt), alpha = exp2f(m - m_new);
                if (i) {
                    ok = __all_sync(0xffffffffu, mbar_wait(odone + 2 * map + ((i - 1) & 1), ((i - 1) >> 1) & 1));
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    for (int c = 0; c < a.vdp; c += 32) {
                        uint32_t o[32];
                        __syncwarp();
                        tmem_ld32(tO + map * vo + lanes + c, o);
                        #pragma unroll
                        for (int j = 0; j < 32; j++) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
                        tmem_st32(tO + map * vo + lanes + c, o);
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
            mbar_arrive(pready + 2 * map + (i & 1));
        }
        ok = __all_sync(0xffffffffu, ok && mbar_wait(odone + 2 * map + ((n_tiles - 1) & 1), ((n_tiles - 1) >> 1) & 1));
        if (!ok) atomicOr(a.err, LG_ERR_MBAR_TIMEOUT | 16384);
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        s_l[map][row] = l;
        asm volatile("bar.sync 1, %0;" :: "n"(MAPS * 128) : "memory");        // both maps' products have finished
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const float c1 = 1.0f / s_l[0][row], c2 = MAPS > 1 ? a.lambda / s_l[MAPS - 1][row] : 0.0f;
        constexpr int KEEP = MAPS > 1 ? 2 : 1;                 // column groups of 32 a thread holds at most (vdp <= 64 MAPS)
        if constexpr (MAPS == 1) {
            for (int c = 0; c < a.vdp; c += 32) {
                uint32_t o[32];
                __syncwarp();
                tmem_ld32(tO + lanes + c, o);
                if (tok >= a.n || !ok) continue;
                uint4 *dst = (uint4 *)((bf16 *)a.out + (size_t)tok * a.ldo + (size_t)h * a.vdp + c);
                #pragma unroll
                for (int j = 0; j < 4; j++)
                    if (c + 8 * j < a.vdp) {
                        auto v = [&](int k) { return __uint_as_float(o[8 * j + k]) * c1; };
                        dst[j] = make_uint4(pack_bf16(v(0), v(1)), pack_bf16(v(2), v(3)), pack_bf16(v(4), v(5)), pack_bf16(v(6), v(7)));
                    }
            }
        } else {
            float o[KEEP][32], ss = 0.0f;
            #pragma unroll
            for (int k = 0; k < KEEP; k++) {
                const int c = (2 * k + map) * 32;              // warps w and w + 4 take the column groups in turn
                #pragma unroll
                for (int j = 0; j < 32; j++) o[k][j] = 0.0f;
                if (c < a.vdp) {
                    uint32_t x[32], y[32];
                    __syncwarp();
                    tmem_ld32(tO + lanes + c, x);
                    tmem_ld32(tO + vo + lanes + c, y);
                    #pragma unroll
                    for (int j = 0; j < 32; j++) {
                        if (c + j < a.vdp) o[k][j] = __uint_as_float(x[j]) * c1 - __uint_as_float(y[j]) * c2;
                        ss = fmaf(o[k][j], o[k][j], ss);
                    }
                }
            }
            s_ss[map][row] = ss;
            asm volatile("bar.sync 1, %0;" :: "n"(MAPS * 128) : "memory");
            const float f = a.out_mult / sqrtf((s_ss[0][row] + s_ss[MAPS - 1][row]) / (float)a.vd + a.eps);
            #pragma unroll
            for (int k = 0; k < KEEP; k++) {
                const int c = (2 * k + map) * 32;
                if (c >= a.vdp || tok >= a.n || !ok) continue;
                uint4 *dst = (uint4 *)((bf16 *)a.out + (size_t)tok * a.ldo + (size_t)h * a.vdp + c);
                #pragma unroll
                for (int j = 0; j < 4; j++)
                    if (c + 8 * j < a.vdp) {
                        auto v = [&](int i) { return o[k][8 * j + i] * f; };
                        dst[j] = make_uint4(pack_bf16(v(0), v(1)), pack_bf16(v(2), v(3)), pack_bf16(v(4), v(5)), pack_bf16(v(6), v(7)));
                    }
            }
        }
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    }
    __syncthreads();
    if (warp == ROWW + 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem), "r"(tcols) : "memory");
    }
}
