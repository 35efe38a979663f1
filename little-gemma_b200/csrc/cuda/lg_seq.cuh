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
// the same in the precision of the element type it ends in
template <typename T> __device__ __forceinline__ float silu_as(float z) { return silu_f(z); }
template <> __device__ __forceinline__ float silu_as<bf16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
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
// with destinations of their own (activation rows, or cache rows in a ring).  Thread: 8 channels x LG_CONV_RUN tokens, whose rows (and
// the filter's history) are all requested before the first is used; the threads of the first run also write the ring, after their
// reads of it.  lg_conv_any_kernel is the same for any number of taps, `run` tokens per thread.
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
#define LG_CONV_RUN 8
// 8 elements as they lie in memory
template <typename T> struct LgRaw8;
template <> struct LgRaw8<float> { float4 a, b; };
template <> struct LgRaw8<bf16> { uint4 a; };
__device__ __forceinline__ void widen8(const LgRaw8<float> &r, float (&f)[8]) { *(float4 *)f = r.a; *(float4 *)(f + 4) = r.b; }
__device__ __forceinline__ void widen8(const LgRaw8<bf16> &r, float (&f)[8]) {
    const uint32_t u[4] = {r.a.x, r.a.y, r.a.z, r.a.w};
    #pragma unroll
    for (int i = 0; i < 4; i++) { const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *)&u[i]); f[2 * i] = x.x; f[2 * i + 1] = x.y; }
}
// the last rows of the block into the ring, by the threads that have read it
template <typename TI, typename T>
__device__ __forceinline__ void conv_keep(const LgConvArgs &a, const TI *src, T *ring, int pos) {
    for (int t = max(0, a.M - (a.mask + 1) / 2); t < a.M; t++) {
        float v[LG_CONV_V];
        load_elems<LG_CONV_V>(src + (size_t)t * a.ld, v);
        store_elems<LG_CONV_V>(ring + (size_t)((pos + t) & a.mask) * a.nch, v);
    }
}
template <typename T> __device__ __forceinline__ T *conv_out(const LgConvArgs &a, int c, LgConvOut &o) {
    o = c < a.o[0].end ? a.o[0] : c < a.o[1].end ? a.o[1] : a.o[2];
    return (T *)o.out + c - (c < a.o[0].end ? 0 : c < a.o[1].end ? a.o[0].end : a.o[1].end);
}
template <typename TI, typename T, int TAPS>
__global__ void __launch_bounds__(LG_CONV_THREADS) lg_conv_kernel(LgConvArgs a) {
    constexpr int V = LG_CONV_V, R = LG_CONV_RUN;
    pdl_launch();
    const int c = (blockIdx.x * LG_CONV_THREADS + threadIdx.x) * V;
    if (c >= a.nch) return;
    float w[TAPS][V], bias[V];
    #pragma unroll
    for (int j = 0; j < TAPS; j++) load_elems<V>(a.w + (size_t)j * a.nch + c, w[j]);
    #pragma unroll
    for (int i = 0; i < V; i++) bias[i] = 0.0f;
    if (a.bias) load_elems<V>(a.bias + c, bias);
    pdl_wait();
    const int pos = *a.pos, t0 = blockIdx.y * R;
    const TI *src = (const TI *)a.src + a.ch0 + c;
    T *ring = (T *)a.ring + c;
    LgRaw8<TI> raw[R];
    #pragma unroll
    for (int t = 0; t < R; t++) if (t0 + t < a.M) raw[t] = *(const LgRaw8<TI> *)(src + (size_t)(t0 + t) * a.ld);
    float u[TAPS][V];                                              // u[j] meets w[j]; the last one is the present
    #pragma unroll
    for (int j = 0; j < TAPS - 1; j++) {
        const int t = t0 - TAPS + 1 + j;
        if (t >= 0) {
            load_elems<V>(src + (size_t)t * a.ld, u[j]);
            #pragma unroll
            for (int i = 0; i < V; i++) u[j][i] = round_elem<T>(u[j][i]);
        } else if (pos + t >= 0) load_elems<V>(ring + (size_t)((pos + t) & a.mask) * a.nch, u[j]);
        else {
            #pragma unroll
            for (int i = 0; i < V; i++) u[j][i] = 0.0f;
        }
    }
    LgConvOut o;
    T *out = conv_out<T>(a, c, o);
    #pragma unroll
    for (int t = 0; t < R; t++) {
        if (t0 + t >= a.M) break;
        widen8(raw[t], u[TAPS - 1]);
        float y[V];
        #pragma unroll
        for (int i = 0; i < V; i++) {
            u[TAPS - 1][i] = round_elem<T>(u[TAPS - 1][i]);
            y[i] = bias[i];
            #pragma unroll
            for (int j = 0; j < TAPS; j++) y[i] = fmaf(w[j][i], u[j][i], y[i]);
            if (a.silu) y[i] = silu_as<T>(y[i]);
            #pragma unroll
            for (int j = 0; j < TAPS - 1; j++) u[j][i] = u[j + 1][i];
        }
        store_elems<V>(out + (size_t)(o.ring_rows ? (pos + t0 + t) % o.ring_rows : t0 + t) * o.ld, y);
    }
    if (blockIdx.y == 0) conv_keep(a, src, ring, pos);
}
template <typename TI, typename T>
__global__ void __launch_bounds__(LG_CONV_THREADS) lg_conv_any_kernel(LgConvArgs a) {
    constexpr int V = LG_CONV_V;
    pdl_launch();
    const int c = (blockIdx.x * LG_CONV_THREADS + threadIdx.x) * V, taps = a.taps;
    if (c >= a.nch) return;
    pdl_wait();
    const int pos = *a.pos, t0 = blockIdx.y * a.run, t1 = min(a.M, t0 + a.run);
    const TI *src = (const TI *)a.src + a.ch0 + c;
    T *ring = (T *)a.ring + c;
    LgConvOut o;
    T *out = conv_out<T>(a, c, o);
    for (int t = t0; t < t1; t++) {
        float y[V];
        #pragma unroll
        for (int i = 0; i < V; i++) y[i] = 0.0f;
        if (a.bias) load_elems<V>(a.bias + c, y);
        for (int j = 0; j < taps; j++) {
            const int s = t - taps + 1 + j;
            if (pos + s < 0) continue;
            float u[V], w[V];
            if (s >= 0) load_elems<V>(src + (size_t)s * a.ld, u); else load_elems<V>(ring + (size_t)((pos + s) & a.mask) * a.nch, u);
            load_elems<V>(a.w + (size_t)j * a.nch + c, w);
            #pragma unroll
            for (int i = 0; i < V; i++) y[i] = fmaf(w[i], round_elem<T>(u[i]), y[i]);
        }
        if (a.silu) {
            #pragma unroll
            for (int i = 0; i < V; i++) y[i] = silu_as<T>(y[i]);
        }
        store_elems<V>(out + (size_t)(o.ring_rows ? (pos + t) % o.ring_rows : t) * o.ld, y);
    }
    if (blockIdx.y == 0) conv_keep(a, src, ring, pos);
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
#define LG_SSM_TC 16                                 // tokens staged at once: by a prompt block, and by a step (whose common case is one
#define LG_SSM_TC_STEP 4                             // replayed and one new token; it is kept small, see the carve-out of the decode step's kernels)
#define LG_SSM_ROWS 16
__host__ __device__ constexpr size_t lg_ssm_step_smem(int taps, int np) { return (size_t)(2 * taps + LG_SSM_TC_STEP) * (2 * np + LG_SSM_ROWS) * 4; }
template <typename T, int NPL, bool WIDE>
__global__ void __launch_bounds__(LG_SSM_THREADS) lg_ssm_step_kernel(LgSsmStepArgs a) {
    constexpr int NS = 32 * NPL, VW = NPL < 4 ? NPL : 4, TC = WIDE ? LG_SSM_TC : LG_SSM_TC_STEP, VR = 4;
    __shared__ __align__(16) float sB[TC][NS], sC[TC][NS];
    __shared__ float sx[TC][LG_SSM_ROWS], sdt[TC], sdec[TC];
    extern __shared__ __align__(16) float ssm_rows[];                // narrow: filters and bias [taps + 1][ncv], raw rows [TC + taps - 1][ncv]
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
    // the channels of this CTA, four at a time: B and C of its group, its value rows
    const int ncv = 2 * a.np + LG_SSM_ROWS, nq = ncv >> 2;
    auto channel = [&](int k) { return k < a.np ? inner + g * a.np + k : k < 2 * a.np ? inner + (a.groups + g) * a.np + k - a.np : h * a.vdp + v0 + k - 2 * a.np; };
    float *raw = ssm_rows + (size_t)(a.taps + 1) * ncv;
    if (!WIDE) {
        load_state();                                // written by an earlier forward
        for (int u = tid; u < (a.taps + 1) * nq; u += LG_SSM_THREADS) {
            const int j = u / nq, k = (u % nq) * 4;
            float4 f = make_float4(0, 0, 0, 0);
            if (j < a.taps) f = *(const float4 *)(a.w + (size_t)j * a.nch + channel(k)); else if (a.bias) f = *(const float4 *)(a.bias + channel(k));
            *(float4 *)(ssm_rows + (size_t)j * ncv + k) = f;
        }
        for (int i = tid; i < TC * (NS - a.np); i += LG_SSM_THREADS) { const int t = i / (NS - a.np), k = a.np + i % (NS - a.np); sB[t][k] = sC[t][k] = 0.0f; }
    }
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
            // staged token t sits at position first + t; raw rows of positions below pos come from the ring, the others go into it
            const float *src = (const float *)a.src;
            T *ring = (T *)a.ring;
            const int first = pos - n_replay + c0, r0 = first - a.taps + 1, nr = nt + a.taps - 1;
            for (int u0 = tid; u0 < nr * nq; u0 += 4 * LG_SSM_THREADS) {
                float f[4][4];
                #pragma unroll
                for (int i = 0; i < 4; i++) {            // four loads in flight before the first store
                    const int u = u0 + i * LG_SSM_THREADS, p = r0 + u / nq, ch = channel((u % nq) * 4);
                    f[i][0] = f[i][1] = f[i][2] = f[i][3] = 0.0f;
                    if (u >= nr * nq) continue;
                    if (p >= pos) load_elems<4>(src + (size_t)(p - pos) * a.ld + a.ch0 + ch, f[i]);
                    else if (p >= 0) load_elems<4>(ring + (size_t)(p & a.mask) * a.nch + ch, f[i]);
                }
                #pragma unroll
                for (int i = 0; i < 4; i++) {
                    const int u = u0 + i * LG_SSM_THREADS, r = u / nq, k = (u % nq) * 4, p = r0 + r;
                    if (u >= nr * nq) continue;
                    if (p >= pos) {
                        if (k >= 2 * a.np || (blockIdx.y == 0 && h == g * per)) store_elems<4>(ring + (size_t)(p & a.mask) * a.nch + channel(k), f[i]);
                        #pragma unroll
                        for (int j = 0; j < 4; j++) f[i][j] = round_elem<T>(f[i][j]);
                    }
                    *(float4 *)(raw + (size_t)r * ncv + k) = *(const float4 *)f[i];
                }
            }
            if (tid < nt) {
                const int p = first + tid;
                const float rdt = p >= pos ? src[(size_t)(p - pos) * a.ld + a.dt_off + h] : a.dt_ring[(size_t)(p & a.mask) * a.heads + h];
                const float dt = softplus_f(rdt + dtb);
                sdt[tid] = dt; sdec[tid] = expf(A * dt);
                if (p >= pos && blockIdx.y == 0) a.dt_ring[(size_t)(p & a.mask) * a.heads + h] = rdt;
            }
            __syncthreads();
            for (int u = tid; u < nt * ncv; u += LG_SSM_THREADS) {
                const int t = u / ncv, k = u % ncv;
                float acc = ssm_rows[(size_t)a.taps * ncv + k];
                for (int j = 0; j < a.taps; j++) acc = fmaf(ssm_rows[(size_t)j * ncv + k], raw[(size_t)(t + j) * ncv + k], acc);
                acc = round_elem<T>(silu_as<T>(acc));
                if (k < a.np) sB[t][k] = acc; else if (k < 2 * a.np) sC[t][k - a.np] = acc; else sx[t][k - 2 * a.np] = acc;
            }
        }
        __syncthreads();
        for (int t = 0; t < nt; t++) {
            if (!WIDE && c0 + t == n_replay && (n_replay || fresh)) store_state();       // the state at pos
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
            if (!WIDE && c0 + t < n_replay) continue;
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
    }
    if (WIDE || a.M == 0) store_state();             // behind the block; (narrow) a replay alone
}

// ---------------------------------------------------------------------------------------------
// gate, then RMS norm of equal parts of a row: out = unit(y * silu(z)) * w
// ---------------------------------------------------------------------------------------------
// Rows are sections of vdp columns per head of which vd count; part g takes elements [g n, (g + 1) n) of the row without padding.
// One CTA per part and token, or (parts of up to 1024 elements) one warp; items of V elements stay in registers between the two passes.
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
            for (int j = 0; j < 4; j++) { f[i][j] = yv[j] * silu_as<TO>(zv[j]); ss = fmaf(f[i][j], f[i][j], ss); }
        } else { f[i][0] = from_elem(y[at]) * silu_as<TO>(from_elem(z[at])); ss = fmaf(f[i][0], f[i][0], ss); }
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
#define LG_GN_WARPS 8
template <typename TI, typename TO, int IPT>
__global__ void __launch_bounds__(LG_GN_WARPS * 32) lg_gated_norm_warp_kernel(LgGatedNormArgs a, int parts, int rows) {
    pdl_launch(); pdl_wait();
    const int job = blockIdx.x * LG_GN_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31, tok = job / parts, part = job % parts;
    if (tok >= rows) return;
    const TI *y = (const TI *)a.y + (size_t)tok * a.ldy, *z = (const TI *)a.z + (size_t)tok * a.ldz;
    float f[IPT][4], zv[IPT][4], ss = 0.0f;
    auto place = [&](int item) {
        const int e = part * a.n + item * 4;
        return a.vd == a.vdp ? e : e / a.vd * a.vdp + e % a.vd;
    };
    #pragma unroll
    for (int i = 0; i < IPT; i++) {
        const int item = lane + i * 32;
        if (item * 4 < a.n) { const int at = place(item); load_elems<4>(y + at, f[i]); load_elems<4>(z + at, zv[i]); }
        else f[i][0] = f[i][1] = f[i][2] = f[i][3] = zv[i][0] = zv[i][1] = zv[i][2] = zv[i][3] = 0.0f;
    }
    #pragma unroll
    for (int i = 0; i < IPT; i++)
        #pragma unroll
        for (int j = 0; j < 4; j++) { f[i][j] *= silu_as<TO>(zv[i][j]); ss = fmaf(f[i][j], f[i][j], ss); }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.n + a.eps);
    TO *out = (TO *)a.out + (size_t)tok * a.ldo;
    #pragma unroll
    for (int i = 0; i < IPT; i++) {
        const int item = lane + i * 32;
        if (item * 4 >= a.n) continue;
        const int at = place(item);
        float wv[4];
        load_elems<4>(a.w + at, wv);
        #pragma unroll
        for (int j = 0; j < 4; j++) wv[j] *= f[i][j] * inv;
        store_elems<4>(out + at, wv);
    }
}
