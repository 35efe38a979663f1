// lg_seq.cuh -- layers that carry state from token to token: short causal convolutions and Mamba-2 (state-space) layers.
//
// Sequence state and positions.  A cache row can be overwritten, a recurrent state cannot be unwound, yet a verify block may be
// cut back to any of its tokens and a step may be repeated.  So the state kept in memory is the one BEFORE the latest narrow block
// (at position `base`), beside a ring of the raw projected rows of the latest positions; the next block, at any position
// base .. base + have, replays the rows in between -- it holds the state in registers anyway -- stores the state it arrives at and
// goes on with its own tokens.  Position 0 starts a new sequence.  A wide (prompt) block leaves the state behind its last token.
//
// Precision: rows and convolution outputs are elements of the mode (bf16 or f32); step sizes, decays, states and sums are f32.
#pragma once
#include "lg_dense.cuh"

struct LgSeqCtl {                   // device-resident, one per cache
    int base, have;                 // position of the stored states; tokens behind it that can be replayed
    int n_replay, fresh;            // of the block being run: tokens to replay (positions base_now .. pos - 1); a new sequence starts
    int pad[12];
};
__device__ __forceinline__ void seq_begin(LgSeqCtl *c, int pos, int m, int wide, int *err) {
    const int d = pos - c->base;
    const bool fresh = pos == 0;
    if (!fresh && (d < 0 || d > c->have)) atomicOr(err, LG_ERR_SEQ_POS);
    c->fresh = fresh;
    c->n_replay = fresh ? 0 : min(max(d, 0), c->have);
    c->base = wide ? pos + m : pos;
    c->have = wide ? 0 : m;
}
__global__ void lg_seq_begin_kernel(LgSeqCtl *c, const int *pos, int m, int wide, int *err) {
    pdl_launch(); pdl_wait();
    if (threadIdx.x == 0) seq_begin(c, *pos, m, wide, err);
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
// through the mode's element type
template <typename T> __device__ __forceinline__ float round_elem(float v) { T o; to_elem(v, o); return from_elem(o); }

// V consecutive elements
template <int V> __device__ __forceinline__ void load_elems(const float *p, float (&f)[V]) {
    #pragma unroll
    for (int i = 0; i < V; i += 4) *(float4 *)(f + i) = *(const float4 *)(p + i);
}
template <int V> __device__ __forceinline__ void load_elems(const bf16 *p, float (&f)[V]) {
    #pragma unroll
    for (int i = 0; i < V; i += 4) {
        const uint2 u = *(const uint2 *)(p + i);
        const float2 a = __bfloat1622float2(*(const __nv_bfloat162 *)&u.x), b = __bfloat1622float2(*(const __nv_bfloat162 *)&u.y);
        f[i] = a.x; f[i + 1] = a.y; f[i + 2] = b.x; f[i + 3] = b.y;
    }
}
template <int V> __device__ __forceinline__ void store_elems(float *p, const float (&f)[V]) {
    #pragma unroll
    for (int i = 0; i < V; i += 4) *(float4 *)(p + i) = *(const float4 *)(f + i);
}
template <int V> __device__ __forceinline__ void store_elems(bf16 *p, const float (&f)[V]) {
    #pragma unroll
    for (int i = 0; i < V; i += 4) *(uint2 *)(p + i) = make_uint2(pack_bf16(f[i], f[i + 1]), pack_bf16(f[i + 2], f[i + 3]));
}

// ---------------------------------------------------------------------------------------------
// short convolution: y[t][c] = bias[c] + sum_j w[j][c] u[t - taps + 1 + j][c], optionally through silu
// ---------------------------------------------------------------------------------------------
// Channels are the columns ch0 .. ch0 + nch of the projection rows; positions before the block come from the ring (row p at
// p & mask, channel-major as in the block), positions before 0 are zeros.  The outputs go to up to three stretches of channels
// with destinations of their own (activation rows, or cache rows in a ring).  Thread: 8 channels x `run` tokens; the threads of
// the first run also write the ring, after their reads of it.
struct LgConvOut { int end; void *out; int ld, ring_rows; };       // channels below `end`; ring_rows 0: row = token, else (pos + token) % ring_rows
struct LgConvArgs {
    const void *src; int ld, ch0, nch;
    const float *w, *bias; int taps;
    void *ring; int mask;
    const int *pos; int M, run, silu;
    LgConvOut o[3];
};
#define LG_CONV_V 8
#define LG_CONV_THREADS 128
template <typename TI, typename T, int TAPS>
__global__ void __launch_bounds__(LG_CONV_THREADS) lg_conv_kernel(LgConvArgs a) {
    constexpr int V = LG_CONV_V, H = TAPS ? TAPS : 16;             // TAPS 0: any number up to 16
    pdl_launch();
    const int c = (blockIdx.x * LG_CONV_THREADS + threadIdx.x) * V, taps = TAPS ? TAPS : a.taps;
    if (c >= a.nch) return;
    float w[H][V], bias[V];
    #pragma unroll
    for (int j = 0; j < H; j++) if (j < taps) load_elems<V>(a.w + (size_t)j * a.nch + c, w[j]);
    #pragma unroll
    for (int i = 0; i < V; i++) bias[i] = 0.0f;
    if (a.bias) load_elems<V>(a.bias + c, bias);
    pdl_wait();
    const int pos = *a.pos, t0 = blockIdx.y * a.run, t1 = min(a.M, t0 + a.run);
    const TI *src = (const TI *)a.src + a.ch0 + c;
    T *ring = (T *)a.ring + c;
    auto fetch = [&](int t, float (&u)[V]) {
        if (t >= 0) {
            load_elems<V>(src + (size_t)t * a.ld, u);
            #pragma unroll
            for (int i = 0; i < V; i++) u[i] = round_elem<T>(u[i]);
        } else if (pos + t >= 0) load_elems<V>(ring + (size_t)((pos + t) & a.mask) * a.nch, u);
        else {
            #pragma unroll
            for (int i = 0; i < V; i++) u[i] = 0.0f;
        }
    };
    const LgConvOut &o = c < a.o[0].end ? a.o[0] : c < a.o[1].end ? a.o[1] : a.o[2];
    const int base = c < a.o[0].end ? 0 : c < a.o[1].end ? a.o[0].end : a.o[1].end;
    T *out = (T *)o.out + (c - base);
    float u[H][V];                                                 // u[j] meets w[j]
    #pragma unroll
    for (int j = 0; j < H - 1; j++) if (j < taps - 1) fetch(t0 - taps + 1 + j, u[j]);
    for (int t = t0; t < t1; t++) {
        float y[V], now[V];
        fetch(t, now);
        #pragma unroll
        for (int i = 0; i < V; i++) y[i] = bias[i];
        #pragma unroll
        for (int j = 0; j < H - 1; j++)
            if (j < taps - 1) {
                #pragma unroll
                for (int i = 0; i < V; i++) y[i] = fmaf(w[j][i], u[j][i], y[i]);
            }
        #pragma unroll
        for (int j = 0; j < H; j++)
            if (j == taps - 1) {
                #pragma unroll
                for (int i = 0; i < V; i++) y[i] = fmaf(w[j][i], now[i], y[i]);
            }
        #pragma unroll
        for (int j = 0; j < H - 1; j++)
            if (j < taps - 1) {
                #pragma unroll
                for (int i = 0; i < V; i++) u[j][i] = j == taps - 2 ? now[i] : u[j + 1 < H ? j + 1 : j][i];
            }
        if (a.silu) {
            #pragma unroll
            for (int i = 0; i < V; i++) y[i] = silu_f(y[i]);
        }
        store_elems<V>(out + (size_t)(o.ring_rows ? (pos + t) % o.ring_rows : t) * o.ld, y);
    }
    if (blockIdx.y == 0)
        for (int t = max(0, a.M - (a.mask + 1) / 2); t < a.M; t++) {
            float v[V];
            load_elems<V>(src + (size_t)t * a.ld, v);
            store_elems<V>(ring + (size_t)((pos + t) & a.mask) * a.nch, v);
        }
}

// ---------------------------------------------------------------------------------------------
// state-space step: the recurrence token by token, the state in registers
// ---------------------------------------------------------------------------------------------
//   S_t = exp(-exp(A_log) dt) S_(t-1) + dt x_t B_t^T,   y_t = S_t C_t + D x_t,   dt = softplus(raw + dt_bias)
// CTA (h, s): value rows 16 s .. of head h; a warp owns 4 rows, its lanes the state columns (NPL each, vectors of up to 4).
// State in memory: [head][vdp][nst] f32, nst = 32 NPL.  WIDE false: up to 8 tokens straight from the projection rows -- the
// convolution, the replay of earlier tokens and the ring are done here, no other kernel stands between the two matmuls.  WIDE
// true: a whole prompt block from convolved rows (32-bit mode, and sizes the chunked kernels do not hold).
struct LgSsmStepArgs {
    const void *src; int ld, ch0, dt_off;            // projection rows; first convolved column; (narrow) column of the raw step sizes
    const float *w, *bias; int taps, nch;            // convolution [taps][nch]; channels: x [heads vdp] | B [groups np] | C [groups np]
    void *ring; float *dt_ring; int mask;
    const float *dt_src; int ld_dt;                  // wide: raw step sizes [token][..]
    const float *dt_bias, *a_log, *d;
    float *state; int heads, vdp, np, groups;
    const LgSeqCtl *ctl; const int *pos; int M;
    int fresh;                                       // wide: a new sequence starts with the block
    void *y; int ldy;                                // narrow: f32 rows; wide: T rows; [token][heads vdp]
};
#define LG_SSM_THREADS 128
#define LG_SSM_TC 16                                 // tokens staged at once: 8 replayed + 8 new
#define LG_SSM_ROWS 16
template <typename T, int NPL, bool WIDE>
__global__ void __launch_bounds__(LG_SSM_THREADS) lg_ssm_step_kernel(LgSsmStepArgs a) {
    constexpr int NS = 32 * NPL, VW = NPL < 4 ? NPL : 4, TC = LG_SSM_TC, VR = 4;
    __shared__ __align__(16) float sB[TC][NS], sC[TC][NS];
    __shared__ float sx[TC][LG_SSM_ROWS], sdt[TC], sdec[TC];
    pdl_launch();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, v0 = blockIdx.y * LG_SSM_ROWS;
    const int per = a.heads / a.groups, g = h / per, inner = a.heads * a.vdp;
    const float dtb = a.dt_bias[h], A = -expf(a.a_log[h]), D = a.d[h];
    // register i of a lane holds column col(i)
    auto col = [&](int i) { return (i / VW) * 32 * VW + lane * VW + i % VW; };
    float *st = a.state + ((size_t)h * a.vdp + v0 + warp * VR) * NS;
    float S[VR][NPL];
    auto load_state = [&]() {
        #pragma unroll
        for (int r = 0; r < VR; r++)
            #pragma unroll
            for (int i = 0; i < NPL; i += VW) {
                const float *p = st + (size_t)r * NS + col(i);
                if (VW == 4) { const float4 f = *(const float4 *)p; S[r][i] = f.x; S[r][i + 1 < NPL ? i + 1 : i] = f.y; S[r][i + 2 < NPL ? i + 2 : i] = f.z; S[r][i + 3 < NPL ? i + 3 : i] = f.w; }
                else for (int j = 0; j < VW; j++) S[r][i + j] = p[j];
            }
    };
    auto store_state = [&]() {
        #pragma unroll
        for (int r = 0; r < VR; r++)
            #pragma unroll
            for (int i = 0; i < NPL; i += VW) {
                float *p = st + (size_t)r * NS + col(i);
                if (VW == 4) *(float4 *)p = make_float4(S[r][i], S[r][i + 1 < NPL ? i + 1 : i], S[r][i + 2 < NPL ? i + 2 : i], S[r][i + 3 < NPL ? i + 3 : i]);
                else for (int j = 0; j < VW; j++) p[j] = S[r][i + j];
            }
    };
    if (!WIDE) load_state();                         // written by an earlier forward
    pdl_wait();
    const int pos = *a.pos;
    const int n_replay = WIDE ? 0 : a.ctl->n_replay;
    const bool fresh = WIDE ? a.fresh != 0 : a.ctl->fresh != 0;
    if (WIDE && !fresh) load_state();
    if (fresh) {
        #pragma unroll
        for (int r = 0; r < VR; r++)
            #pragma unroll
            for (int i = 0; i < NPL; i++) S[r][i] = 0.0f;
    }
    if (!WIDE && n_replay == 0 && a.M == 0) {        // nothing between the stored state and here
        if (fresh) store_state();
        return;
    }
    const int total = n_replay + a.M;
    for (int c0 = 0; c0 < total; c0 += TC) {
        const int nt = min(TC, total - c0);
        if (c0) __syncthreads();
        if (WIDE) {
            const T *src = (const T *)a.src;
            for (int u = tid; u < nt * (2 * NS + LG_SSM_ROWS); u += LG_SSM_THREADS) {
                const int t = u / (2 * NS + LG_SSM_ROWS), k = u % (2 * NS + LG_SSM_ROWS);
                const T *row = src + (size_t)(c0 + t) * a.ld;
                if (k < NS) sB[t][k] = k < a.np ? from_elem(row[inner + g * a.np + k]) : 0.0f;
                else if (k < 2 * NS) sC[t][k - NS] = k - NS < a.np ? from_elem(row[inner + (a.groups + g) * a.np + k - NS]) : 0.0f;
                else sx[t][k - 2 * NS] = from_elem(row[h * a.vdp + v0 + k - 2 * NS]);
            }
            if (tid < nt) {
                const float dt = softplus_f(a.dt_src[(size_t)(c0 + tid) * a.ld_dt + h] + dtb);
                sdt[tid] = dt; sdec[tid] = expf(A * dt);
            }
        } else {
            // staged token t sits at position first + t; raw rows of positions below pos come from the ring
            const float *src = (const float *)a.src;
            T *ring = (T *)a.ring;
            const int first = pos - n_replay;
            for (int k = tid; k < 2 * NS + LG_SSM_ROWS; k += LG_SSM_THREADS) {
                int ch = -1;
                bool writer = true;                  // of this channel's rows in the ring
                if (k < NS) { if (k < a.np) ch = inner + g * a.np + k; }
                else if (k < 2 * NS) { if (k - NS < a.np) ch = inner + (a.groups + g) * a.np + k - NS; }
                else ch = h * a.vdp + v0 + k - 2 * NS;
                if (k < 2 * NS) writer = blockIdx.y == 0 && h == g * per;
                float *dst = k < NS ? &sB[0][k] : k < 2 * NS ? &sC[0][k - NS] : &sx[0][k - 2 * NS];
                const int ldd = k < 2 * NS ? NS : LG_SSM_ROWS;
                if (ch < 0) { for (int t = 0; t < nt; t++) dst[t * ldd] = 0.0f; continue; }
                const float b = a.bias ? a.bias[ch] : 0.0f;
                for (int t = 0; t < nt; t++) {
                    float acc = b;
                    for (int j = 0; j < a.taps; j++) {
                        const int p = first + t - a.taps + 1 + j;
                        float u = 0.0f;
                        if (p >= pos) u = round_elem<T>(src[(size_t)(p - pos) * a.ld + a.ch0 + ch]);
                        else if (p >= 0) u = from_elem(ring[(size_t)(p & a.mask) * a.nch + ch]);
                        acc = fmaf(a.w[(size_t)j * a.nch + ch], u, acc);
                    }
                    dst[t * ldd] = round_elem<T>(silu_f(acc));
                }
                if (writer)
                    for (int t = 0; t < a.M; t++) to_elem(src[(size_t)t * a.ld + a.ch0 + ch], ring[(size_t)((pos + t) & a.mask) * a.nch + ch]);
            }
            if (tid < nt) {
                const int p = first + tid;
                const float raw = p >= pos ? src[(size_t)(p - pos) * a.ld + a.dt_off + h] : a.dt_ring[(size_t)(p & a.mask) * a.heads + h];
                const float dt = softplus_f(raw + dtb);
                sdt[tid] = dt; sdec[tid] = expf(A * dt);
                if (p >= pos && blockIdx.y == 0) a.dt_ring[(size_t)(p & a.mask) * a.heads + h] = raw;
            }
        }
        __syncthreads();
        for (int t = 0; t < nt; t++) {
            if (!WIDE && t == n_replay && (n_replay || fresh)) store_state();       // the state at pos
            const float dt = sdt[t], dec = sdec[t];
            float dx[VR], y[VR];
            #pragma unroll
            for (int r = 0; r < VR; r++) { dx[r] = dt * sx[t][warp * VR + r]; y[r] = 0.0f; }
            #pragma unroll
            for (int i = 0; i < NPL; i += VW) {
                float b[VW], c[VW];
                if (VW == 4) { *(float4 *)b = *(const float4 *)&sB[t][col(i)]; *(float4 *)c = *(const float4 *)&sC[t][col(i)]; }
                else for (int j = 0; j < VW; j++) { b[j] = sB[t][col(i) + j]; c[j] = sC[t][col(i) + j]; }
                #pragma unroll
                for (int r = 0; r < VR; r++)
                    #pragma unroll
                    for (int j = 0; j < VW; j++) {
                        S[r][i + j] = fmaf(dec, S[r][i + j], dx[r] * b[j]);
                        y[r] = fmaf(S[r][i + j], c[j], y[r]);
                    }
            }
            if (!WIDE && t < n_replay) continue;
            #pragma unroll
            for (int r = 0; r < VR; r++) y[r] = warp_sum(y[r]);
            float out = y[0];
            #pragma unroll
            for (int r = 1; r < VR; r++) if (lane == r) out = y[r];
            if (lane < VR) {
                const int v = warp * VR + lane;
                const float o = fmaf(D, sx[t][v], out);
                const size_t at = (size_t)(c0 + t - n_replay) * a.ldy + h * a.vdp + v0 + v;
                if (WIDE) to_elem(o, ((T *)a.y)[at]); else ((float *)a.y)[at] = o;
            }
        }
        if (!WIDE && a.M == 0) store_state();        // replay only
    }
    if (WIDE) store_state();
}

// ---------------------------------------------------------------------------------------------
// gate, then RMS norm of equal parts of a row: out = unit(y * silu(z)) * w
// ---------------------------------------------------------------------------------------------
// Rows are sections of vdp columns per head of which vd count; part g takes elements [g n, (g + 1) n) of the row without padding.
// One CTA per part and token; items of V elements stay in registers between the two passes.
struct LgGatedNormArgs {
    const void *y, *z; int ldy, ldz;
    const float *w;                      // [heads vdp]
    int vd, vdp, n; float eps;
    void *out; int ldo;
};
template <typename TI, typename TO, int V, int IPT>
__global__ void lg_gated_norm_kernel(LgGatedNormArgs a) {
    __shared__ float red[32];
    pdl_launch(); pdl_wait();
    const TI *y = (const TI *)a.y + (size_t)blockIdx.y * a.ldy, *z = (const TI *)a.z + (size_t)blockIdx.y * a.ldz;
    float f[IPT][V];
    float ss = 0.0f;
    auto place = [&](int item) {
        const int e = blockIdx.x * a.n + item * V;
        return a.vd == a.vdp ? e : e / a.vd * a.vdp + e % a.vd;
    };
    #pragma unroll
    for (int i = 0; i < IPT; i++) {
        const int item = threadIdx.x + i * blockDim.x;
        if (item * V >= a.n) continue;
        const int at = place(item);
        if constexpr (V == 4) {
            float yv[4], zv[4];
            load_elems<4>(y + at, yv); load_elems<4>(z + at, zv);
            #pragma unroll
            for (int j = 0; j < 4; j++) { f[i][j] = yv[j] * silu_f(zv[j]); ss = fmaf(f[i][j], f[i][j], ss); }
        } else { f[i][0] = from_elem(y[at]) * silu_f(from_elem(z[at])); ss = fmaf(f[i][0], f[i][0], ss); }
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)a.n + a.eps);
    TO *out = (TO *)a.out + (size_t)blockIdx.y * a.ldo;
    #pragma unroll
    for (int i = 0; i < IPT; i++) {
        const int item = threadIdx.x + i * blockDim.x;
        if (item * V >= a.n) continue;
        const int at = place(item);
        if constexpr (V == 4) {
            float wv[4], o[4];
            load_elems<4>(a.w + at, wv);
            #pragma unroll
            for (int j = 0; j < 4; j++) o[j] = f[i][j] * inv * wv[j];
            store_elems<4>(out + at, o);
        } else to_elem(f[i][0] * inv * a.w[at], out[at]);
    }
}
