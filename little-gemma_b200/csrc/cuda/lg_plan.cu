// lg_plan.cu -- the family of models described by a layer plan (lg_plan.h): dense bf16 weights, per-layer mixers (latent attention,
// grouped windowed attention, state-space), f32 residual rows.  Decode and verify steps run the small-M matmuls, the split attention
// over the cache and the state-space step; prompts run blocks of up to PLAN_BLOCK tokens through the tcgen05 matmul, block attention
// and chunked state-space kernels.  In 32-bit mode every product, activation and cache row is f32.
#include <algorithm>
#include <tuple>
#include "lg_engine.h"
#include "lg_plan.h"
#include "lg_latent.cuh"
#include "lg_seq.cuh"
#include "lg_ssd.cuh"
#include "lg_window.cuh"

namespace lg {

constexpr int PLAN_BLOCK = 2048;              // tokens of one wide block
constexpr int PLAN_HEAD_ROWS = 128;           // logits rows made at once behind a wide block
constexpr size_t PLAN_SMEM_MAX = 227 * 1024;          // dynamic shared memory of a CTA: all of it, and what kernels with static arrays ask for
constexpr size_t PLAN_SMEM_SMALL = 200 * 1024;

inline int up(int v, int m) { return (v + m - 1) / m * m; }

// A dense matrix on the device: [rows_alloc][ldk], zero beyond its rows and columns.
struct DMat {
    void *w = nullptr;
    int rows = 0, k = 0, ldk = 0, rows_alloc = 0;             // rows: a multiple of 32
    CUtensorMap map[2];                                       // bf16: boxes of 128 and of 256 rows
};

struct PlanLayer {
    struct lg_plan_layer p;
    int dimp, rotp, kvp, vdp, ffp, ldc;                       // sizes padded to whole 16-element groups; ldc: cache row
    int kv_off, rot_off, g_off;                               // columns of the input projection's row: [query latent | latent | key part | gate]
    int owns, spec;                                           // spec: which rotation table
    int rt;                                                   // row tiles of 16 per CTA of the decode attention (0: the row kernel)
    DMat in, uq, ukT, uk, uv, o, gu, down;             // uk: keys from latents (prompt pass); ukT: the same per head, transposed (decode)
    // grouped attention and state-space layers (lg_plan_seq.cuh)
    int np = 0, npl = 0, nst = 0, vs = 0;                     // state columns padded to 16; per lane of the step kernel; of a stored state row; value columns per chunk CTA
    int in_rows = 0, ch0 = 0, nch = 0, dt_off = 0, q_cols = 0, k_cols = 0;   // projection row: [q | k | v] or [z | x | B | C | step sizes]; convolved columns ch0 .. ch0 + nch
    int at_cols = 0, act_off = 0, mask = 0, C = 1;            // output product's columns: mixer rows, feed-forward rows from act_off on; ring of projected rows; key splits
    int chunked = 1;                                          // the prompt kernels hold the sizes
    float lambda = 0.0f, out_mult = 1.0f, eps = 0.0f;
    float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *d = nullptr, *gnorm = nullptr;
    DMat inup;                                                // input projection over the feed-forward's; `in` and `gu` are its parts
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *q_norm = nullptr, *kv_norm = nullptr, *sink = nullptr;
};

// Activations of up to `cap` token rows.
struct PlanBuf {
    int cap = 0;
    float *x = nullptr, *pj = nullptr, *o = nullptr, *gu = nullptr;
    void *h = nullptr, *cq = nullptr, *q = nullptr, *qa = nullptr, *ol = nullptr, *at = nullptr, *act = nullptr;
    void *h2 = nullptr, *cv = nullptr, *y = nullptr;          // second norm; convolved rows; state-space outputs
    float *dt = nullptr; bf16 *s_hi = nullptr, *s_lo = nullptr;    // raw step sizes; states before every chunk
    std::vector<float2 *> tab;
    int *toks = nullptr, *pos = nullptr;                      // of the block (narrow: the engine's round state)
};

struct PlanModel {
    struct lg_plan *plan = nullptr;
    std::vector<PlanLayer> L;
    DMat embed;
    float *out_norm = nullptr;
    struct Rot { float base; int dims; double *freq; };
    std::vector<Rot> rot;
    struct Run { int layer, slot; const float *step; };       // a looped layer runs once per pass, with cache and state of its own
    std::vector<Run> runs;
    float *step = nullptr;                                    // [times][width]
    const struct kvcache *st_kv = nullptr; int st_lo = -1, st_hi = -1;       // positions a block may start at, as far as the host knows (-1: ask the device)
    PlanBuf nb, wb;
    bool wide_ok = false;
    // bound to a cache
    int max_seq = 0, seq_alloc = 0, C = 1;
    float *part = nullptr; float2 *part_ml = nullptr;
    bf16 *kx = nullptr, *vx = nullptr;                       // one layer's expanded keys [position][H dimp] and values [H vdp][position]
    int *want = nullptr; void *hg = nullptr; float *wlog = nullptr;
    float *logits = nullptr;                                  // 32-bit: rows of a head without F_LOGITS
    std::map<std::tuple<const void *, int, int, int, int>, CUtensorMap> maps;
};

// ------------------------------------------------------------------------------------------
// loading
// ------------------------------------------------------------------------------------------
const struct gguf_tensor *need(Engine *e, int L, const char *leaf, int rows, int cols) {
    char name[96];
    snprintf(name, sizeof name, "%s.weight", leaf);
    const struct gguf_tensor *t = find_t(e->ctx, L, name);
    if (!t) { fprintf(stderr, "lg_b200: layer %d: tensor %s is missing from the model\n", L, leaf); exit(1); }
    if ((int)t->dims[0] != (cols ? cols : rows) || (int)t->dims[1] != (cols ? rows : 1)) {
        fprintf(stderr, "lg_b200: %s is %d x %d, expected %d x %d\n", t->name, (int)t->dims[1], (int)t->dims[0], cols ? rows : 1, cols ? cols : rows);
        exit(1);
    }
    if (t->type != GGML_TYPE_BF16 && t->type != GGML_TYPE_F32 && t->type != GGML_TYPE_F16) {
        fprintf(stderr, "lg_b200: %s: layer-plan models have dense weights (bf16, f16, f32), not ggml type %u\n", t->name, t->type);
        exit(1);
    }
    return t;
}
std::vector<float> row_f32(const struct gguf_tensor *t, int row) {
    const size_t n = (size_t)t->dims[0];
    std::vector<float> f(n);
    dequantize_into(t->type, (const uint8_t *)t->data + (size_t)row * n * (t->type == GGML_TYPE_F32 ? 4 : 2), f.data(), (int64_t)n);
    return f;
}
float *vec(Engine *e, int L, const char *leaf, int n) { return upload_f32(row_f32(need(e, L, leaf, n, 0), 0).data(), (size_t)n); }

uint16_t bf16_bits(float f) {
    uint32_t u;
    memcpy(&u, &f, 4);
    return (uint16_t)((u + 0x7fff + ((u >> 16) & 1)) >> 16);
}

// A matrix under construction on the host, in the element type of the engine's mode.
struct MatBuild {
    bool f32; int rows, k, ldk;
    std::vector<uint8_t> buf;
    MatBuild(Engine *e, int rows_, int k_) : f32(e->f32), rows(up(rows_, 32)), k(k_), ldk(up(k_, 64)) { buf.assign((size_t)rows * ldk * (f32 ? 4 : 2), 0); }
    void put(size_t i, float v) {
        if (f32) memcpy(&buf[i * 4], &v, 4);
        else { const uint16_t b = bf16_bits(v); memcpy(&buf[i * 2], &b, 2); }
    }
    // row `src` of t; its columns come in segments of seg that start every seg_to columns here (0: one piece)
    void row(int dst, const struct gguf_tensor *t, int src, int seg = 0, int seg_to = 0, int col0 = 0) {
        const int n = (int)t->dims[0];
        if (!f32 && t->type == GGML_TYPE_BF16 && seg == seg_to) {
            memcpy(&buf[((size_t)dst * ldk + col0) * 2], (const uint8_t *)t->data + (size_t)src * n * 2, (size_t)n * 2);
            return;
        }
        const std::vector<float> f = row_f32(t, src);
        for (int i = 0; i < n; i++) put((size_t)dst * ldk + col0 + (seg ? i / seg * seg_to + i % seg : i), f[i]);
    }
    DMat upload(Engine *e) {
        DMat m;
        m.rows = rows; m.k = k; m.ldk = ldk; m.rows_alloc = up(rows, 256);
        const size_t es = f32 ? 4 : 2;
        m.w = dalloc<uint8_t>((size_t)m.rows_alloc * ldk * es);
        h2d_sync(m.w, buf.data(), buf.size());
        e->weight_bytes += (size_t)rows * k * es;
        if (!f32)
            for (int i = 0; i < 2; i++) m.map[i] = tiled_map(m.w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, ldk, m.rows_alloc, (long long)ldk * 2, DN_GEMM_BK, 128 << i);
        return m;
    }
};

// `groups` groups of `rows` rows of t, each padded to `to` rows; rows of group g start at g * t_stride
void put_groups(MatBuild &b, int dst0, const struct gguf_tensor *t, int groups, int rows, int to) {
    for (int g = 0; g < groups; g++)
        for (int r = 0; r < rows; r++) b.row(dst0 + g * to + r, t, g * rows + r);
}

template <typename K> void smem_attr(K kernel, size_t bytes = PLAN_SMEM_MAX) { LG_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes)); }
template <int EPI, bool RMSX> void gemv_attrs() {
    smem_attr(lg_dn_gemv_kernel<EPI, 1, RMSX>, PLAN_SMEM_SMALL); smem_attr(lg_dn_gemv_kernel<EPI, 2, RMSX>, PLAN_SMEM_SMALL);
    smem_attr(lg_dn_gemv_kernel<EPI, 4, RMSX>, PLAN_SMEM_SMALL); smem_attr(lg_dn_gemv_kernel<EPI, 8, RMSX>, PLAN_SMEM_SMALL);
}
void seq_attributes();
void plan_attributes() {
    static bool done[64] = {false};
    int dev = 0;
    LG_CHECK(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 64 || done[dev]) return;
    done[dev] = true;
    gemv_attrs<DN_STORE, true>();
    smem_attr(lg_dn_gemm_kernel<128, DN_G_F32>, dn_gemm_smem<128>()); smem_attr(lg_dn_gemm_kernel<256, DN_G_F32>, dn_gemm_smem<256>());
    smem_attr(lg_dn_gemm_kernel<128, DN_G_BF16>, dn_gemm_smem<128>()); smem_attr(lg_dn_gemm_kernel<256, DN_G_BF16>, dn_gemm_smem<256>());
    smem_attr(lg_dn_gemm_kernel<128, DN_G_GLU>, dn_gemm_smem<128>()); smem_attr(lg_dn_gemm_kernel<256, DN_G_GLU>, dn_gemm_smem<256>());
    smem_attr(lg_latent_dec_attn_kernel<1, 2>); smem_attr(lg_latent_dec_attn_kernel<1, 4>); smem_attr(lg_latent_dec_attn_kernel<1, 8>);
    smem_attr(lg_latent_dec_attn_kernel<2, 2>); smem_attr(lg_latent_dec_attn_kernel<2, 4>); smem_attr(lg_latent_dec_attn_kernel<2, 8>);
    smem_attr(lg_latent_pf_attn_kernel);
    seq_attributes();
    smem_attr(lg_latent_merge_kernel, PLAN_SMEM_SMALL); smem_attr(lg_latent_attn_rows_kernel<float>, PLAN_SMEM_SMALL); smem_attr(lg_latent_attn_rows_kernel<bf16>, PLAN_SMEM_SMALL);
}

void seq_buf_alloc(Engine *e, PlanBuf &b, int cap, bool narrow);
void buf_alloc(Engine *e, PlanBuf &b, int cap, bool narrow) {
    PlanModel *pm = e->plan;
    if (pm->plan->form == LG_FORM_PARALLEL) { seq_buf_alloc(e, b, cap, narrow); return; }
    const size_t es = e->f32 ? 4 : 2;
    size_t pj = 0, o = up(pm->plan->width, 32), gu = 0, cq = 0, q = 0, qa = 0, ol = 0, at = 0, act = 0;
    for (auto &l : pm->L) {
        const size_t H = l.p.heads;
        pj = std::max(pj, (size_t)l.in.rows); cq = std::max(cq, (size_t)l.uq.ldk);
        q = std::max(q, (size_t)up((int)H * (l.dimp + l.rotp), 32));
        qa = std::max(qa, H * l.ldc); ol = std::max(ol, H * l.kvp); at = std::max(at, (size_t)l.o.ldk);
        if (l.p.ff) { act = std::max(act, (size_t)l.down.ldk); gu = std::max(gu, (size_t)l.gu.rows); }
    }
    auto elems = [&](size_t per) { return (void *)dalloc<uint8_t>(((size_t)cap * per + 256) * es); };
    b.cap = cap;
    b.x = narrow ? e->x : dalloc<float>((size_t)cap * pm->plan->width);
    b.pj = dalloc<float>(cap * pj); b.o = dalloc<float>(cap * o);
    if (e->f32) b.gu = dalloc<float>(cap * gu + 16);
    b.h = elems(up(pm->plan->width, 64)); b.cq = elems(cq); b.q = elems(q); b.at = elems(at); b.act = elems(act + 64);
    if (narrow || e->f32) { b.qa = elems(qa); b.ol = elems(ol); }
    for (auto &r : pm->rot) b.tab.push_back(dalloc<float2>((size_t)cap * (r.dims / 2) + 1));
    if (!narrow) { b.toks = nullptr; b.pos = dalloc<int>(1); }
}
void buf_free(PlanBuf &b, bool narrow) {
    if (!narrow) cudaFree(b.x);
    cudaFree(b.pj); cudaFree(b.o); cudaFree(b.gu); cudaFree(b.h); cudaFree(b.cq); cudaFree(b.q); cudaFree(b.qa); cudaFree(b.ol); cudaFree(b.at); cudaFree(b.act);
    cudaFree(b.h2); cudaFree(b.cv); cudaFree(b.y); cudaFree(b.dt); cudaFree(b.s_hi); cudaFree(b.s_lo);
    for (auto t : b.tab) cudaFree(t);
    cudaFree(b.toks); cudaFree(b.pos);
    b = PlanBuf();
}

void layer_sizes(PlanLayer &l) {
    const struct lg_plan_layer &p = l.p;
    l.dimp = up(p.dim, 16); l.rotp = up(p.rot_dim, 16); l.kvp = up(p.kv_rank, 16); l.vdp = up(p.vdim, 16); l.ffp = up(p.ff, 16);
    l.ldc = l.kvp + l.rotp;
}

void seq_layer_sizes(PlanLayer &l);
void seq_layer_load(Engine *e, int L, PlanLayer &l);
void seq_layer_free(PlanLayer &l);
float *vec_offset(Engine *e, int L, const char *leaf, int n, float offset);

void latent_layer_load(Engine *e, int i, PlanLayer &l) {
    PlanModel *pm = e->plan;
    const int W = pm->plan->width;
    layer_sizes(l);
    const struct lg_plan_layer &p = l.p;
    const int H = p.heads;
    l.owns = p.kv_src == i;
    l.kv_off = up(p.q_rank, 16);
    l.rot_off = l.kv_off + (l.owns ? l.kvp : 0);
    l.g_off = l.rot_off + (l.owns ? l.rotp : 0);
    {   // everything that reads the layer's input: query latent, cached latent and key part, output gate
        MatBuild b(e, l.g_off + H * l.vdp, W);
        put_groups(b, 0, need(e, i, "attn_q_a", p.q_rank, W), 1, p.q_rank, 0);
        if (l.owns) {
            const struct gguf_tensor *t = need(e, i, "attn_kv_a", p.kv_rank + p.rot_dim, W);
            for (int r = 0; r < p.kv_rank + p.rot_dim; r++) b.row(r < p.kv_rank ? l.kv_off + r : l.rot_off + r - p.kv_rank, t, r);
        }
        put_groups(b, l.g_off, need(e, i, "attn_gate", H * p.vdim, W), H, p.vdim, l.vdp);
        l.in = b.upload(e);
    }
    {   // queries: per head [unrotated | rotated]
        const struct gguf_tensor *t = need(e, i, "attn_q_b", H * (p.dim + p.rot_dim), p.q_rank);
        MatBuild b(e, H * (l.dimp + l.rotp), p.q_rank);
        for (int h = 0; h < H; h++)
            for (int r = 0; r < p.dim + p.rot_dim; r++)
                b.row(h * (l.dimp + l.rotp) + (r < p.dim ? r : l.dimp + r - p.dim), t, h * (p.dim + p.rot_dim) + r);
        l.uq = b.upload(e);
    }
    const struct gguf_tensor *uk = need(e, i, "attn_k_b", H * p.dim, p.kv_rank), *uv = need(e, i, "attn_v_b", H * p.vdim, p.kv_rank);
    {   // the key expansion transposed per head: rows = latent columns, contraction over the head's dimensions
        MatBuild b(e, H * l.kvp, p.dim);
        for (int h = 0; h < H; h++)
            for (int d = 0; d < p.dim; d++) {
                const std::vector<float> f = row_f32(uk, h * p.dim + d);
                for (int r = 0; r < p.kv_rank; r++) b.put((size_t)(h * l.kvp + r) * b.ldk + d, f[r]);
            }
        l.ukT = b.upload(e);
    }
    {
        MatBuild b(e, H * l.vdp, p.kv_rank);
        put_groups(b, 0, uv, H, p.vdim, l.vdp);
        l.uv = b.upload(e);
    }
    if (!e->f32) {
        MatBuild b(e, H * l.dimp, p.kv_rank);
        put_groups(b, 0, uk, H, p.dim, l.dimp);
        const size_t before = e->weight_bytes;
        l.uk = b.upload(e);
        e->weight_bytes = before;                        // a second copy of weights already counted
    }
    {
        const struct gguf_tensor *t = need(e, i, "attn_output", W, H * p.vdim);
        MatBuild b(e, W, H * l.vdp);
        for (int r = 0; r < W; r++) b.row(r, t, r, p.vdim, l.vdp);
        l.o = b.upload(e);
    }
    if (p.ff) {
        const struct gguf_tensor *g = need(e, i, "ffn_gate", p.ff, W), *u = need(e, i, "ffn_up", p.ff, W), *d = need(e, i, "ffn_down", W, p.ff);
        MatBuild b(e, 2 * l.ffp, W);
        for (int r = 0; r < p.ff; r++) { b.row(r / 8 * 16 + r % 8, g, r); b.row(r / 8 * 16 + 8 + r % 8, u, r); }   // 8 gate rows, their 8 up rows
        l.gu = b.upload(e);
        MatBuild c(e, W, l.ffp);
        for (int r = 0; r < W; r++) c.row(r, d, r);
        l.down = c.upload(e);
        l.norm2 = vec(e, i, "ffn_norm", W); l.norm2b = vec(e, i, "post_ffw_norm", W);
    }
    l.norm1 = vec(e, i, "attn_norm", W); l.norm1b = vec(e, i, "post_attention_norm", W);
    l.q_norm = vec(e, i, "attn_q_a_norm", p.q_rank);
    if (l.owns) l.kv_norm = vec(e, i, "attn_kv_a_norm", p.kv_rank);
    l.sink = vec(e, i, "attn_sinks", H);
    l.spec = -1;
    for (size_t s = 0; s < pm->rot.size(); s++) if (pm->rot[s].base == p.rot_base && pm->rot[s].dims == p.rot_dims) l.spec = (int)s;
    if (l.spec < 0) {
        std::vector<double> f(p.rot_dims / 2 + 1);
        for (int j = 0; j < p.rot_dims / 2; j++) f[j] = pow((double)p.rot_base, -2.0 * j / p.rot_dims);
        double *d = dalloc<double>(f.size());
        h2d_sync(d, f.data(), f.size() * 8);
        l.spec = (int)pm->rot.size();
        pm->rot.push_back({p.rot_base, p.rot_dims, d});
    }
    l.rt = l.kvp > 512 ? 0 : lg_latent_dec_smem(2, l.ldc) <= PLAN_SMEM_MAX ? 2 : lg_latent_dec_smem(1, l.ldc) <= PLAN_SMEM_MAX ? 1 : 0;
    if (e->f32) l.rt = 0;
    if (l.vdp > 256 || lg_latent_pf_smem(l.dimp, l.rotp, l.vdp) > PLAN_SMEM_MAX) pm->wide_ok = false;
    if ((size_t)(l.ldc + l.kvp + 128) * 4 > PLAN_SMEM_SMALL || (size_t)LG_LM_GROUPS * l.kvp * 4 > PLAN_SMEM_SMALL ||
        (size_t)LG_MAXM * (l.uq.ldk + 8) * 2 > PLAN_SMEM_SMALL) { fprintf(stderr, "lg_b200: layer %d: latent sizes beyond what the kernels hold\n", i); exit(1); }
}

void plan_load(Engine *e) {
    PlanModel *pm = e->plan = new PlanModel();
    plan_attributes();
    pm->plan = lg_plan_read(e->ctx);
    if (!pm->plan) exit(1);
    const struct lg_plan *P = pm->plan;
    const int W = P->width;
    if (W > 16 * 1024) { fprintf(stderr, "lg_b200: rows of %d elements exceed the norm kernel's 16384\n", W); exit(1); }
    pm->L.resize(P->n_layer);
    pm->wide_ok = true;
    for (int i = 0; i < P->n_layer; i++) {
        PlanLayer &l = pm->L[i];
        l.p = P->layer[i];
        l.eps = P->norm_eps;
        if (P->form == LG_FORM_PARALLEL) { seq_layer_sizes(l); seq_layer_load(e, i, l); }
        else latent_layer_load(e, i, l);
    }
    if (e->f32) pm->wide_ok = true;
    static const int wide = env_int("LG_PREFILL_WIDE", 1);
    if (!wide) pm->wide_ok = false;
    {
        const struct gguf_tensor *t = need(e, -1, "token_embd", P->vocab, W);
        MatBuild b(e, P->vocab, W);
        for (int r = 0; r < P->vocab; r++) b.row(r, t, r);
        pm->embed = b.upload(e);
    }
    e->head.ldo = pm->embed.rows;
    pm->out_norm = vec_offset(e, -1, "output_norm", W, P->norm_offset);
    if (P->loop_times) {
        const struct gguf_tensor *t = need(e, -1, "loop_step", P->loop_times, W);
        std::vector<float> f;
        for (int r = 0; r < P->loop_times; r++) { const std::vector<float> row = row_f32(t, r); f.insert(f.end(), row.begin(), row.end()); }
        pm->step = upload_f32(f.data(), f.size());
    }
    for (int r = 0; r < lg_plan_runs(P); r++) {
        int pass = -1;
        const int L = lg_plan_run_layer(P, r, &pass);
        pm->runs.push_back({L, r, pass < 0 ? nullptr : pm->step + (size_t)pass * W});
    }
    buf_alloc(e, pm->nb, LG_MAXM, true);
    if (e->f32) pm->logits = dalloc<float>((size_t)LG_MAXM * e->head.ldo);
}

void dmat_free(DMat &m) { cudaFree(m.w); m = DMat(); }
void plan_unbind(PlanModel *pm) {
    cudaFree(pm->part); cudaFree(pm->part_ml); cudaFree(pm->kx); cudaFree(pm->vx); cudaFree(pm->want); cudaFree(pm->hg); cudaFree(pm->wlog);
    pm->part = nullptr; pm->part_ml = nullptr; pm->kx = pm->vx = nullptr; pm->want = nullptr; pm->hg = nullptr; pm->wlog = nullptr;
    if (pm->wb.cap) buf_free(pm->wb, false);
    pm->maps.clear();
}
void plan_release(Engine *e) {
    PlanModel *pm = e->plan;
    if (!pm) return;
    plan_unbind(pm);
    for (auto &l : pm->L) {
        if (l.inup.w) l.in = l.gu = DMat();                  // parts of it
        for (DMat *m : {&l.in, &l.uq, &l.ukT, &l.uk, &l.uv, &l.o, &l.gu, &l.down, &l.inup}) dmat_free(*m);
        seq_layer_free(l);
        for (float *v : {l.norm1, l.norm1b, l.norm2, l.norm2b, l.q_norm, l.kv_norm, l.sink}) cudaFree(v);
    }
    for (auto &r : pm->rot) cudaFree(r.freq);
    dmat_free(pm->embed);
    cudaFree(pm->out_norm); cudaFree(pm->logits); cudaFree(pm->step);
    buf_free(pm->nb, true);
    lg_plan_free(pm->plan);
    delete pm;
    e->plan = nullptr;
}

// ------------------------------------------------------------------------------------------
// cache
// ------------------------------------------------------------------------------------------
int cache_rows(int max_seq) { return up(max_seq, 128); }      // whole boxes of the tiled copies

int plan_kv_slots(const struct model *m) {
    struct lg_plan *P = lg_plan_read(m->ctx);
    const int n = P ? lg_plan_runs(P) : 0;
    lg_plan_free(P);
    return n;
}
int seq_kv_init(struct kvcache *kv, const struct lg_plan *P, bool f32);
int plan_kv_init(struct kvcache *kv, const struct model *m, bool f32) {
    struct lg_plan *P = lg_plan_read(m->ctx);
    if (!P) return -1;
    if (P->form == LG_FORM_PARALLEL) {
        const int rc = seq_kv_init(kv, P, f32);
        lg_plan_free(P);
        return rc;
    }
    for (int i = 0; i < P->n_layer; i++) {
        PlanLayer l;
        l.p = P->layer[i];
        layer_sizes(l);
        kv->kv_dim[i] = l.ldc;
        kv->f16[i] = f32 ? 0 : 2;
        if (l.p.kv_src != i) continue;                        // borrows the rows of an earlier layer
        kv->seq[i] = kv->max_seq;
        const size_t bytes = (size_t)cache_rows(kv->max_seq) * l.ldc * (f32 ? 4 : 2);
        LG_CHECK(cudaMalloc(&kv->k[i], bytes));
        LG_CHECK(cudaMemset(kv->k[i], 0, bytes));
    }
    lg_plan_free(P);
    return 0;
}

int latent_splits(const Engine *e, int heads, int max_seq);
void seq_bind(Engine *e, const struct kvcache *kv);
void plan_bind(Engine *e, const struct kvcache *kv) {
    PlanModel *pm = e->plan;
    plan_unbind(pm);
    pm->max_seq = kv->max_seq; pm->seq_alloc = cache_rows(kv->max_seq);
    if (pm->plan->form == LG_FORM_PARALLEL) { seq_bind(e, kv); return; }
    if (e->f32) return;
    size_t rows = 0;
    int most = 1;
    for (auto &l : pm->L) {
        most = std::max(most, l.p.heads);
        rows = std::max(rows, (size_t)l.p.heads * LG_MAXM * l.kvp);
    }
    pm->C = latent_splits(e, most, kv->max_seq);
    size_t heads = 0;
    for (auto &l : pm->L) heads = std::max(heads, (size_t)l.p.heads);
    pm->part = dalloc<float>(rows * pm->C);
    pm->part_ml = dalloc<float2>(heads * LG_MAXM * pm->C);
}

// ------------------------------------------------------------------------------------------
// matmul launches
// ------------------------------------------------------------------------------------------
// Slices of k per 16-row tile: enough warps to keep every SM's loads in flight, at least two chunks of 32 columns each.  A
// property of the matrix alone: it fixes the order in which a row's products are added.
int gemv_ks(const Engine *e, const DMat &W) {
    const int tiles = W.rows / 16, nchunk = W.ldk / 32;
    int ks = 1;
    while (ks < 8 && tiles * ks < e->sm_count * 16 && nchunk / (ks * 2) >= 2) ks *= 2;
    return ks;
}
template <int EPI, bool RMSX>
int launch_dn_gemv(Engine *e, const DMat &W, LgDnGemvArgs a, int groups = 0, int cap_ctas = 1 << 20) {
    a.w = (const bf16 *)W.w; a.ldk = W.ldk; a.n_tiles = groups ? groups * a.tiles_per_group : W.rows / 16;   // (rows behind the last group are padding)
    const int ks = gemv_ks(e, W), tpc = 8 / ks;
    a.n_main = std::min((a.n_tiles + tpc - 1) / tpc, cap_ctas);
    const dim3 grid(a.n_main + (a.job ? a.M : 0));
    const size_t sm = RMSX ? (size_t)a.M * (W.ldk + 8) * 2 : 0;
    switch (ks) {
    case 1: launch_k(e, lg_dn_gemv_kernel<EPI, 1, RMSX>, grid, dim3(DN_GEMV_THREADS), sm, a); break;
    case 2: launch_k(e, lg_dn_gemv_kernel<EPI, 2, RMSX>, grid, dim3(DN_GEMV_THREADS), sm, a); break;
    case 4: launch_k(e, lg_dn_gemv_kernel<EPI, 4, RMSX>, grid, dim3(DN_GEMV_THREADS), sm, a); break;
    default: launch_k(e, lg_dn_gemv_kernel<EPI, 8, RMSX>, grid, dim3(DN_GEMV_THREADS), sm, a); break;
    }
    return a.n_main;
}
// descriptor of a bf16 activation buffer [rows][ld], of which k columns count; made once per buffer, shape and box
const CUtensorMap &buf_map(PlanModel *pm, const void *x, int k, int ld, int rows, int box_r) {
    const auto key = std::make_tuple(x, k, ld, rows, box_r);
    auto it = pm->maps.find(key);
    if (it == pm->maps.end())
        it = pm->maps.emplace(key, tiled_map(x, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, std::min(k, ld), rows, (long long)ld * 2, DN_GEMM_BK, box_r)).first;
    return it->second;
}
// out[i][j] = row i of x (n of them count) . row j of w (w_rows, a multiple of 32); maps of w with boxes of 128 / 256 rows
template <int EPI>
void launch_gemm_maps(Engine *e, const CUtensorMap &x, int n, const CUtensorMap &w128, const CUtensorMap &w256, int w_rows, int nkb, void *out, int ldo, bool w_early, LgDnGemmArgs a = LgDnGemmArgs{}) {
    a.nkb = nkb; a.n_tok = n; a.cols = w_rows; a.out = out; a.ldo = ldo; a.err = e->err; a.w_early = w_early;
    const int ty = (n + DN_GEMM_BM - 1) / DN_GEMM_BM;
    if ((w_rows + 255) / 256 * ty >= e->sm_count)
        launch_k(e, lg_dn_gemm_kernel<256, EPI>, dim3((w_rows + 255) / 256, ty), dim3(DN_GEMM_THREADS), dn_gemm_smem<256>(), x, w256, a);
    else
        launch_k(e, lg_dn_gemm_kernel<128, EPI>, dim3((w_rows + 127) / 128, ty), dim3(DN_GEMM_THREADS), dn_gemm_smem<128>(), x, w128, a);
}
// x: [x_rows][ldx] bf16, of which n rows count
template <int EPI>
void launch_dn_gemm(Engine *e, const DMat &W, const void *x, int ldx, int x_rows, int n, void *out, int ldo, LgDnGemmArgs a = LgDnGemmArgs{}) {
    launch_gemm_maps<EPI>(e, buf_map(e->plan, x, W.k, ldx, x_rows, DN_GEMM_BM), n, W.map[0], W.map[1], W.rows, W.ldk / DN_GEMM_BK, out, ldo, true, a);
}
void launch_f32(Engine *e, const DMat &W, const void *x, int ldx, int n, void *out, int ldo, int groups = 1, int group_rows = 0, int x_group = 0, int out_group = 0, float scale = 1.0f) {
    LgDnF32Args a{};
    a.out_scale = scale;
    a.w = (const float *)W.w; a.ldk = W.ldk; a.rows = groups > 1 ? group_rows : W.rows; a.k = W.k;
    if (groups == 1 && group_rows) a.rows = group_rows;
    a.x = (const float *)x; a.ldx = ldx; a.n = n; a.out = (float *)out; a.ldo = ldo;
    a.w_group = (size_t)group_rows * W.ldk; a.x_group = x_group; a.out_group = out_group;
    launch_k(e, lg_dn_gemm_f32_kernel, dim3((a.rows + 63) / 64, (n + 63) / 64, groups), dim3(256), 0, a);
}

void launch_row_norm(Engine *e, int n, LgRowNormArgs a) {
    // a few elements per thread: barriers among few warps for one row, whole cache lines per warp for many
    const int vec = a.n % 4 == 0 && a.ldx % 4 == 0 && a.ldy % 4 == 0 && a.ld_add % 4 == 0 ? 4 : 1, items = a.n / vec;
    const int threads = std::min(1024, std::max(64, up((items + 1) / 2, 32)));
    const int ipt = (items + threads - 1) / threads;
    auto go = [&](auto kernel) { launch_k(e, kernel, dim3(n), dim3(threads), 0, a); };
    if (e->f32) {
        if (vec == 4) { if (ipt <= 2) go(lg_row_norm_kernel<float, 2, 4>); else go(lg_row_norm_kernel<float, 4, 4>); }
        else go(lg_row_norm_kernel<float, 16, 1>);
    } else {
        if (vec == 4) { if (ipt <= 2) go(lg_row_norm_kernel<bf16, 2, 4>); else go(lg_row_norm_kernel<bf16, 4, 4>); }
        else go(lg_row_norm_kernel<bf16, 16, 1>);
    }
}

void launch_row_norm_par(Engine *e, int n, LgRowNormArgs a) {
    const int vec = a.n % 4 == 0 && a.ldx % 4 == 0 && a.ldy % 4 == 0 && a.ld_add % 4 == 0 ? 4 : 1, items = a.n / vec;
    const int threads = std::min(1024, std::max(64, up((items + 1) / 2, 32)));
    const int ipt = (items + threads - 1) / threads;
    auto go = [&](auto kernel) { launch_k(e, kernel, dim3(n), dim3(threads), 0, a); };
    if (e->f32) {
        if (vec == 4) { if (ipt <= 2) go(lg_row_norm_kernel<float, 2, 4, true>); else go(lg_row_norm_kernel<float, 4, 4, true>); }
        else go(lg_row_norm_kernel<float, 16, 1, true>);
    } else {
        if (vec == 4) { if (ipt <= 2) go(lg_row_norm_kernel<bf16, 2, 4, true>); else go(lg_row_norm_kernel<bf16, 4, 4, true>); }
        else go(lg_row_norm_kernel<bf16, 16, 1, true>);
    }
}

// ------------------------------------------------------------------------------------------
// a pass over the layers
// ------------------------------------------------------------------------------------------
struct Pass {
    PlanBuf *b;
    int n; bool wide;
    const int *toks, *pos;                        // device
    int pos0;                                     // wide: the host's copy of *pos
    bool first = true;                            // wide: the first block of a prompt pass
};

void plan_embed_rows(Engine *e, const int *toks, int n, float *x) {
    const DMat &E = e->plan->embed;
    const int W = e->plan->plan->width;
    if (e->f32) launch_k(e, lg_dn_embed_rows<float>, dim3(n), dim3(256), 0, (const float *)E.w, E.ldk, e->plan->plan->vocab, toks, x, W);
    else launch_k(e, lg_dn_embed_rows<bf16>, dim3(n), dim3(256), 0, (const bf16 *)E.w, E.ldk, e->plan->plan->vocab, toks, x, W);
}

// Splits of the decode attention: as many CTAs as there are SMs for the row tiles of one token, a property of the cache length
// and the head count alone (never of the block's width or the position).
int latent_splits(const Engine *e, int heads, int max_seq) {
    return std::max(1, std::min({e->sm_count / ((heads + 15) / 16), (max_seq + LG_LD_S - 1) / LG_LD_S, LG_LM_MAXC}));
}
void launch_latent_rows(Engine *e, const PlanLayer &l, int n, const LgLatentRowsArgs &a) {
    const size_t sm = (size_t)(l.ldc + l.kvp + 128) * 4;
    if (e->f32) launch_k(e, lg_latent_attn_rows_kernel<float>, dim3(l.p.heads, n), dim3(128), sm, a);
    else launch_k(e, lg_latent_attn_rows_kernel<bf16>, dim3(l.p.heads, n), dim3(128), sm, a);
}
// absorbed queries q [n * H][ldc] over the cache -> latent rows out [n * H][kvp]
void launch_latent_dec(Engine *e, const PlanLayer &l, int n, const void *q, const void *cache, const int *pos, void *out) {
    PlanModel *pm = e->plan;
    const int H = l.p.heads;
    LgLatentDecArgs a{};
    const CUtensorMap &cm = buf_map(pm, cache, l.ldc, l.ldc, pm->seq_alloc, LG_LD_S);
    a.q = (const bf16 *)q; a.ldc = l.ldc; a.kvp = l.kvp; a.rows = n * H; a.H = H;
    a.scale = l.p.scale; a.pos = pos; a.part = pm->part; a.part_ml = pm->part_ml; a.err = e->err;
    const int rt = n * H > 64 ? l.rt : 1;                      // few rows: a row tile per CTA; the arithmetic of a row is the same
    const dim3 grid(pm->C, (n * H + 16 * rt - 1) / (16 * rt)), block(LG_LD_THREADS);
    const size_t sm = lg_latent_dec_smem(rt, l.ldc);
    if (rt == 2) {
        if (l.kvp <= 128) launch_k(e, lg_latent_dec_attn_kernel<2, 2>, grid, block, sm, cm, a);
        else if (l.kvp <= 256) launch_k(e, lg_latent_dec_attn_kernel<2, 4>, grid, block, sm, cm, a);
        else launch_k(e, lg_latent_dec_attn_kernel<2, 8>, grid, block, sm, cm, a);
    } else {
        if (l.kvp <= 128) launch_k(e, lg_latent_dec_attn_kernel<1, 2>, grid, block, sm, cm, a);
        else if (l.kvp <= 256) launch_k(e, lg_latent_dec_attn_kernel<1, 4>, grid, block, sm, cm, a);
        else launch_k(e, lg_latent_dec_attn_kernel<1, 8>, grid, block, sm, cm, a);
    }
    LgLatentMergeArgs m{};
    m.part = pm->part; m.part_ml = pm->part_ml; m.rows = n * H; m.H = H; m.kvp = l.kvp; m.C = pm->C; m.sink = l.sink; m.pos = pos; m.out = (bf16 *)out;
    launch_k(e, lg_latent_merge_kernel, dim3(n * H), dim3(LG_LM_THREADS), (size_t)LG_LM_GROUPS * l.kvp * 4, m);
}
// rotated queries q [n][ldq] over the expanded keys and values of the block's context -> gated rows out [n][ldo]
void launch_latent_prompt(Engine *e, const PlanLayer &l, int n, int q_rows, const void *q, int ldq, const void *cache, const float *gate, int ldg,
                          const int *pos, void *out, int ldo) {
    PlanModel *pm = e->plan;
    LgLatentPfArgs a{};
    a.H = l.p.heads; a.dimp = l.dimp; a.rotp = l.rotp; a.vdp = l.vdp; a.n = n; a.rot_at = l.kvp; a.scale = l.p.scale; a.sink = l.sink;
    a.gate = gate; a.ldg = ldg; a.pos = pos; a.out = (bf16 *)out; a.ldo = ldo; a.err = e->err;
    launch_k(e, lg_latent_pf_attn_kernel, dim3((n + LG_LP_Q - 1) / LG_LP_Q, l.p.heads), dim3(LG_LP_THREADS), lg_latent_pf_smem(l.dimp, l.rotp, l.vdp),
             buf_map(pm, q, ldq, ldq, q_rows, LG_LP_Q), buf_map(pm, pm->kx, l.uk.rows, l.uk.rows, pm->seq_alloc, LG_LP_S),
             buf_map(pm, cache, l.ldc, l.ldc, pm->seq_alloc, LG_LP_S), buf_map(pm, pm->vx, pm->seq_alloc, pm->seq_alloc, l.uv.rows, l.vdp), a);
}

void latent_attention(Engine *e, const struct kvcache *kv, PlanLayer &l, const Pass &p, int only) {
    PlanModel *pm = e->plan;
    PlanBuf &b = *p.b;
    const int H = l.p.heads, n = p.n, qh = l.dimp + l.rotp, ldq = up(H * qh, 32), ld_at = l.o.ldk;
    const float eps = pm->plan->norm_eps;
    void *cache = kv->k[l.p.kv_src];
    const float *gate = b.pj + l.g_off;
    LgCacheRow cr{};
    cr.src = b.pj; cr.ld = l.in.rows; cr.kv_off = l.kv_off; cr.rot_off = l.rot_off; cr.norm_w = l.kv_norm; cr.eps = eps;
    cr.kv_rank = l.p.kv_rank; cr.rot_dim = l.p.rot_dim; cr.rot_dims = l.p.rot_dims; cr.tab = b.tab[l.spec];
    cr.cache = cache; cr.ldc = l.ldc; cr.rot_at = l.kvp; cr.pos = p.pos;
    LgRotQ rq{};
    rq.q = b.q; rq.ldq = ldq; rq.head_stride = qh; rq.rot_at_q = l.dimp; rq.out = b.qa; rq.ldc = l.ldc; rq.rot_at = l.kvp;
    rq.H = H; rq.rot_dim = l.p.rot_dim; rq.rot_dims = l.p.rot_dims; rq.tab = b.tab[l.spec];
    LgLatentPrepArgs pa{};
    pa.src = b.pj; pa.ld = l.in.rows; pa.q_off = 0; pa.q_rank = l.p.q_rank; pa.q_norm = l.q_norm; pa.eps = eps;
    pa.cq = b.cq; pa.ldcq = l.uq.ldk; pa.owns = l.owns; pa.cr = cr;
    LgLatentRowsArgs ra{};
    ra.q = b.qa; ra.cache = cache; ra.ldc = l.ldc; ra.kvp = l.kvp; ra.H = H; ra.sink = l.sink; ra.scale = l.p.scale; ra.pos = p.pos; ra.out = b.ol;

    if (e->f32) {
        launch_k(e, lg_latent_prep_kernel<float>, dim3(n), dim3(128), 0, pa);
        launch_f32(e, l.uq, b.cq, l.uq.ldk, n, b.q, ldq);
        launch_f32(e, l.ukT, b.q, ldq, n, b.qa, H * l.ldc, H, l.kvp, qh, l.ldc);
        launch_k(e, lg_latent_rot_q_kernel<float>, dim3(1, n), dim3(128), 0, rq);
        launch_latent_rows(e, l, n, ra);
        launch_f32(e, l.uv, b.ol, H * l.kvp, n, b.at, ld_at, H, l.vdp, l.kvp, l.vdp);
        launch_k(e, lg_dn_gate_rows, dim3((H * l.vdp + 255) / 256, n), dim3(256), 0, (float *)b.at, ld_at, gate, l.in.rows, H * l.vdp);
        return;
    }
    if (p.wide) {
        const int keys = p.pos0 + n;
        if (only & C_MISC) launch_k(e, lg_latent_prep_kernel<bf16>, dim3(n), dim3(128), 0, pa);
        if (only & C_QKV) launch_dn_gemm<DN_G_BF16>(e, l.uq, b.cq, l.uq.ldk, b.cap, n, b.q, ldq);
        if (only & C_MISC) {
            rq.out = b.q;
            launch_k(e, lg_latent_rot_rows_kernel, dim3((unsigned)std::min(16, (H * l.p.rot_dims / 2 + 127) / 128 + 1), n), dim3(128), 0, rq);
        }
        if (only & C_PLE) {                        // keys [position][H dimp], values transposed [H vdp][position]
            launch_dn_gemm<DN_G_BF16>(e, l.uk, cache, l.ldc, pm->seq_alloc, keys, pm->kx, l.uk.rows);
            launch_gemm_maps<DN_G_BF16>(e, l.uv.map[0], H * l.vdp, buf_map(pm, cache, l.p.kv_rank, l.ldc, pm->seq_alloc, 128),
                                        buf_map(pm, cache, l.p.kv_rank, l.ldc, pm->seq_alloc, 256), up(keys, 32), l.uv.ldk / DN_GEMM_BK, pm->vx, pm->seq_alloc, false);
        }
        if (only & C_ATTN) launch_latent_prompt(e, l, n, b.cap, b.q, ldq, cache, gate, l.in.rows, p.pos, b.at, ld_at);
        return;
    }
    if (only & C_QKV) {
        LgDnGemvArgs q{};                          // normed query latent -> queries; beside it, the cache rows
        q.xf = b.pj; q.ldxf = l.in.rows; q.kx = l.p.q_rank; q.rms_w = l.q_norm; q.eps = eps; q.M = n; q.outh = (bf16 *)b.q; q.ldoh = ldq;
        if (l.owns) { q.job = DN_JOB_CACHE_ROW; q.cr = cr; }
        launch_dn_gemv<DN_STORE, true>(e, l.uq, q);
        LgDnGemvArgs k{};                          // per head onto the latent; beside it, the rotated parts
        k.x = (const bf16 *)b.q; k.ldx = ldq; k.tiles_per_group = l.kvp / 16; k.x_group = qh; k.out_group = l.ldc; k.M = n;
        k.outh = (bf16 *)b.qa; k.ldoh = H * l.ldc; k.job = DN_JOB_ROT_Q; k.rq = rq;
        launch_dn_gemv<DN_STORE, false>(e, l.ukT, k, H);
    }
    if (only & C_ATTN) {
        if (l.rt) launch_latent_dec(e, l, n, b.qa, cache, p.pos, b.ol);
        else launch_latent_rows(e, l, n, ra);
    }
    if (only & C_O) {
        LgDnGemvArgs v{};                          // latent outputs -> gated head values
        v.x = (const bf16 *)b.ol; v.ldx = H * l.kvp; v.tiles_per_group = l.vdp / 16; v.x_group = l.kvp; v.out_group = l.vdp; v.M = n;
        v.outh = (bf16 *)b.at; v.ldoh = ld_at; v.gate = gate; v.ld_gate = l.in.rows;
        launch_dn_gemv<DN_SIGMOID_GATE, false>(e, l.uv, v, H);
    }
}

// out (f32 rows) = W x
void project(Engine *e, const DMat &W, const void *x, int ldx, const Pass &p, float *out) {
    if (e->f32) launch_f32(e, W, x, ldx, p.n, out, W.rows);
    else if (p.wide) launch_dn_gemm<DN_G_F32>(e, W, x, ldx, p.b->cap, p.n, out, W.rows);
    else {
        LgDnGemvArgs a{};
        a.x = (const bf16 *)x; a.ldx = ldx; a.M = p.n; a.out = out; a.ldo = W.rows;
        launch_dn_gemv<DN_STORE, false>(e, W, a);
    }
}
// rows of W x through the gated unit of a feed-forward
void gated(Engine *e, PlanLayer &l, const void *x, int ldx, const Pass &p) {
    PlanBuf &b = *p.b;
    if (e->f32) {
        launch_f32(e, l.gu, x, ldx, p.n, b.gu, l.gu.rows);
        launch_k(e, lg_dn_glu_rows, dim3((l.ffp + 255) / 256, p.n), dim3(256), 0, (const float *)b.gu, l.gu.rows, l.ffp, (float *)b.act, l.down.ldk);
    } else if (p.wide) launch_dn_gemm<DN_G_GLU>(e, l.gu, x, ldx, b.cap, p.n, b.act, l.down.ldk);
    else {
        LgDnGemvArgs a{};
        a.x = (const bf16 *)x; a.ldx = ldx; a.M = p.n; a.outh = (bf16 *)b.act; a.ldoh = l.down.ldk;
        launch_dn_gemv<DN_GLU, false>(e, l.gu, a);
    }
}

#include "lg_plan_seq.cuh"

// x in place -> every layer -> (with final_norm) the normed rows in b->h and, narrow, in e->hidden
void plan_layers(Engine *e, const struct kvcache *kv, const Pass &p, bool final_norm, int only) {
    PlanModel *pm = e->plan;
    PlanBuf &b = *p.b;
    const struct lg_plan *P = pm->plan;
    const int W = P->width, ldh = up(W, 64);
    if (P->form == LG_FORM_PARALLEL) { seq_layers(e, kv, p, final_norm, only); return; }
    if (only & C_MISC)
        for (size_t s0 = 0; s0 < pm->rot.size(); s0 += 8) {
            LgRotTables a{};
            const int ns = (int)std::min(pm->rot.size() - s0, (size_t)8);
            int half = 1;
            for (int i = 0; i < ns; i++) { a.s[i] = {pm->rot[s0 + i].freq, pm->rot[s0 + i].dims / 2, b.tab[s0 + i]}; half = std::max(half, a.s[i].half); }
            a.pos = p.pos; a.n_tok = p.n;
            launch_k(e, lg_dn_rot_tables, dim3((unsigned)std::min(592, (p.n * half + 127) / 128), ns), dim3(128), 0, a);
        }
    LgRowNormArgs r{};
    r.x = b.x; r.ldx = W; r.n = W; r.eps = P->norm_eps; r.center = P->norm_kind == LG_NORM_LAYER; r.mult = P->residual_mult;
    r.y = b.h; r.ldy = ldh;
    r.norm_w = pm->L[0].norm1;
    if (only & C_NORM) launch_row_norm(e, p.n, r);
    r.add = b.o;
    for (int i = 0; i < P->n_layer; i++) {
        PlanLayer &l = pm->L[i];
        const bool last = i + 1 == P->n_layer;
        float *next = last ? (final_norm ? pm->out_norm : nullptr) : pm->L[i + 1].norm1;
        auto resid = [&](const float *add_w, const float *norm_w, bool end) {
            r.add_w = add_w; r.norm_w = norm_w; r.ld_add = l.o.rows;
            r.yf = end && last && final_norm && !p.wide ? e->hidden : nullptr; r.ldyf = W;
            if (only & C_NORM) launch_row_norm(e, p.n, r);
        };
        if (only & C_QKV) project(e, l.in, b.h, ldh, p, b.pj);
        latent_attention(e, kv, l, p, only);
        if (only & C_O) project(e, l.o, b.at, l.o.ldk, p, b.o);
        resid(l.norm1b, l.p.ff ? l.norm2 : next, !l.p.ff);
        if (!l.p.ff) continue;
        if (only & C_GATEUP) gated(e, l, b.h, ldh, p);
        if (only & C_DOWN) project(e, l.down, b.act, l.down.ldk, p, b.o);
        resid(l.norm2b, next, true);
    }
}

void plan_embed(Engine *e, int M) { plan_embed_rows(e, e->st->toks, M, e->x); }

int plan_forward(Engine *e, const struct kvcache *kv, int M, int flags, int only) {
    PlanModel *pm = e->plan;
    if ((only & C_MISC) && !(flags & F_NOEMBED)) plan_embed(e, M);
    Pass p{&pm->nb, M, false, e->st->toks, &e->st->pos, 0};
    plan_layers(e, kv, p, flags & F_HEAD, only);
    if (e->mid_event) LG_CHECK(cudaEventRecord(e->mid_event, e->stream));
    if (!(flags & F_HEAD) || !(only & C_HEAD)) return 1;
    float *lg = flags & F_LOGITS ? e->logits : nullptr;
    const int ldh = up(pm->plan->width, 64);
    if (e->f32) {
        if (!lg) lg = pm->logits;
        launch_f32(e, pm->embed, pm->nb.h, ldh, M, lg, e->head.ldo, 1, 0, 0, 0, pm->plan->logit_scale);
        launch_k(e, lg_dn_argmax_rows, dim3(32, M), dim3(256), 0, (const float *)lg, e->head.ldo, pm->plan->vocab, e->amax_val, e->amax_idx);
        return 32;
    }
    LgDnGemvArgs a{};
    a.x = (const bf16 *)pm->nb.h; a.ldx = ldh; a.M = M; a.rows = pm->plan->vocab; a.out = lg; a.ldo = e->head.ldo;
    a.amax_val = e->amax_val; a.amax_idx = e->amax_idx; a.out_scale = pm->plan->logit_scale;
    return launch_dn_gemv<DN_HEAD, false>(e, pm->embed, a, 0, e->head_ctas);
}

// buffers of the wide pass, at its first use
bool wide_ready(Engine *e) {
    PlanModel *pm = e->plan;
    if (!pm->wide_ok) return false;
    if (pm->wb.cap) return true;
    const int cap = std::max(128, std::min(PLAN_BLOCK, pm->seq_alloc));
    buf_alloc(e, pm->wb, cap, false);
    pm->wb.toks = dalloc<int>(pm->seq_alloc);
    pm->want = dalloc<int>(pm->seq_alloc);
    const int ldh = up(pm->plan->width, 64);
    pm->hg = dalloc<uint8_t>((size_t)PLAN_HEAD_ROWS * ldh * (e->f32 ? 4 : 2));
    pm->wlog = dalloc<float>((size_t)PLAN_HEAD_ROWS * pm->embed.rows);
    if (pm->plan->form == LG_FORM_PARALLEL) return true;
    size_t kx = 0, vx = 0;
    for (auto &l : pm->L) { kx = std::max(kx, (size_t)l.uk.rows); vx = std::max(vx, (size_t)l.uv.rows); }
    if (!e->f32) { pm->kx = dalloc<bf16>((size_t)pm->seq_alloc * kx); pm->vx = dalloc<bf16>((size_t)pm->seq_alloc * vx); }
    return true;
}

int plan_prefill(Engine *e, const struct kvcache *kv, const int *toks, int n, int pos0, const int *want, int n_want, float *logits) {
    PlanModel *pm = e->plan;
    if (!wide_ready(e)) return 0;
    PlanBuf &b = pm->wb;
    const int V = pm->plan->vocab, ldh = up(pm->plan->width, 64), row_bytes = ldh * (e->f32 ? 4 : 2);
    std::vector<int> rel(n_want), starts;
    int i = 0, w = 0;
    for (int k = 0; k < n_want; k++) rel[k] = want[k] % b.cap;
    LG_CHECK(cudaMemcpyAsync(b.toks, toks, (size_t)n * 4, cudaMemcpyHostToDevice, e->stream));
    if (n_want) LG_CHECK(cudaMemcpyAsync(pm->want, rel.data(), (size_t)n_want * 4, cudaMemcpyHostToDevice, e->stream));
    starts.reserve(n / b.cap + 1);
    while (n - i > LG_MAXM) {                                // a last stretch of <= 8 tokens goes through the verify path
        const int m = std::min(b.cap, n - i);
        starts.push_back(pos0 + i);
        LG_CHECK(cudaMemcpyAsync(b.pos, &starts.back(), 4, cudaMemcpyHostToDevice, e->stream));
        Pass p{&b, m, true, b.toks + i, b.pos, pos0 + i, i == 0};
        int hi = w;
        while (hi < n_want && want[hi] < i + m) hi++;
        plan_embed_rows(e, p.toks, m, b.x);
        plan_layers(e, kv, p, hi > w, C_ALL);
        for (; w < hi; w += PLAN_HEAD_ROWS) {
            const int c = std::min(PLAN_HEAD_ROWS, hi - w);
            launch_k(e, lg_dn_gather_rows, dim3(c), dim3(128), 0, (const void *)b.h, (const int *)(pm->want + w), pm->hg, row_bytes);
            if (e->f32) launch_f32(e, pm->embed, pm->hg, ldh, c, pm->wlog, pm->embed.rows, 1, 0, 0, 0, pm->plan->logit_scale);
            else {
                LgDnGemmArgs g{};
                g.out_scale = pm->plan->logit_scale;
                launch_dn_gemm<DN_G_F32>(e, pm->embed, pm->hg, ldh, PLAN_HEAD_ROWS, c, pm->wlog, pm->embed.rows, g);
            }
            LG_CHECK(cudaMemcpy2DAsync(logits + (size_t)w * V, (size_t)V * 4, pm->wlog, (size_t)pm->embed.rows * 4, (size_t)V * 4, c, cudaMemcpyDeviceToHost, e->stream));
        }
        w = hi;
        i += m;
    }
    check_err(e);
    return i;
}

int plan_bench_block(Engine *e, const struct kvcache *kv, int n, int pos0, int only) {
    PlanModel *pm = e->plan;
    if (!wide_ready(e) || n > pm->wb.cap || pos0 + n > kv->max_seq) return -1;
    LG_CHECK(cudaMemsetAsync(pm->wb.pos, 0, 4, e->stream));
    Pass p{&pm->wb, n, true, pm->wb.toks, pm->wb.pos, 0};
    if (only & C_MISC) plan_embed_rows(e, p.toks, n, pm->wb.x);
    plan_layers(e, kv, p, false, only);
    return 0;
}

const LgFamily plan_family = {"layer plan", plan_load, plan_release, plan_kv_slots, plan_kv_init, plan_bind, plan_forward, plan_embed, plan_prefill, plan_bench_block,
                              plan_start, plan_prefix};

}  // namespace lg

extern "C" const lg::LgFamily *lg_family_for(const struct gguf_context *ctx) { return lg_plan_present(ctx) ? &lg::plan_family : nullptr; }

// ==========================================================================================
// kernel-level entry points of the parity tests (host buffers in, host buffers out)
// ==========================================================================================
namespace lg {

// an engine without a model: stream, status word, launch settings, and the descriptor store of the launch helpers
struct Scratch {
    Engine e;
    PlanModel pm;
    std::vector<void *> mem;
    explicit Scratch(bool f32) {
        plan_attributes();
        int dev = 0;
        LG_CHECK(cudaGetDevice(&dev));
        LG_CHECK(cudaDeviceGetAttribute(&e.sm_count, cudaDevAttrMultiProcessorCount, dev));
        LG_CHECK(cudaStreamCreateWithFlags(&e.stream, cudaStreamNonBlocking));
        e.err = dalloc<int>(1); mem.push_back(e.err);
        e.f32 = f32; e.plan = &pm;
    }
    ~Scratch() {
        cudaStreamSynchronize(e.stream);
        for (void *p : mem) cudaFree(p);
        cudaStreamDestroy(e.stream);
    }
    size_t es() const { return e.f32 ? 4 : 2; }
    // rows x n f32 values as [rows_alloc][ld] elements of the mode's type (plus slack), zero elsewhere
    void *rows(const float *src, int rows, int n, int rows_alloc, int ld) {
        std::vector<uint8_t> h(((size_t)rows_alloc * ld + 256) * es(), 0);
        for (int r = 0; r < rows; r++)
            for (int i = 0; i < n; i++) {
                const float v = src[(size_t)r * n + i];
                if (e.f32) memcpy(&h[((size_t)r * ld + i) * 4], &v, 4);
                else { const uint16_t b = bf16_bits(v); memcpy(&h[((size_t)r * ld + i) * 2], &b, 2); }
            }
        void *d = dalloc<uint8_t>(h.size());
        h2d_sync(d, h.data(), h.size());
        mem.push_back(d);
        return d;
    }
    template <typename T> T *put(const T *src, size_t n) {
        T *d = dalloc<T>(n);
        if (src) h2d_sync(d, src, n * sizeof(T));
        mem.push_back(d);
        return d;
    }
    // n elements of a device buffer, as f32
    std::vector<float> get(const void *d, size_t n, bool f32) {
        std::vector<float> out(n);
        check_err(&e);
        if (f32) { LG_CHECK(cudaMemcpy(out.data(), d, n * 4, cudaMemcpyDeviceToHost)); return out; }
        std::vector<uint16_t> b(n);
        LG_CHECK(cudaMemcpy(b.data(), d, n * 2, cudaMemcpyDeviceToHost));
        for (size_t i = 0; i < n; i++) { const uint32_t u = (uint32_t)b[i] << 16; memcpy(&out[i], &u, 4); }
        return out;
    }
};

}  // namespace lg

using namespace lg;

extern "C" int lg_dense_matmul_host(const float *w, const float *w_up, int m, int k, const float *x, int n, int f32, float *out) {
    if (m < 1 || k < 1 || n < 1 || (w_up && m % 8)) return -1;
    Scratch s(f32 != 0);
    Engine *e = &s.e;
    MatBuild b(e, w_up ? 2 * up(m, 16) : m, k);
    for (int r = 0; r < m; r++)
        for (int i = 0; i < k; i++) {
            b.put((size_t)(w_up ? r / 8 * 16 + r % 8 : r) * b.ldk + i, w[(size_t)r * k + i]);
            if (w_up) b.put((size_t)(r / 8 * 16 + 8 + r % 8) * b.ldk + i, w_up[(size_t)r * k + i]);
        }
    DMat W = b.upload(e);
    s.mem.push_back(W.w);
    const int xr = up(n, 128);
    PlanLayer l;
    l.gu = W; l.ffp = up(m, 16); l.down.ldk = up(l.ffp, 64);
    s.pm.nb.cap = xr;
    s.pm.nb.gu = s.put<float>(nullptr, (size_t)xr * W.rows);
    s.pm.nb.act = s.put<uint8_t>(nullptr, ((size_t)xr * l.down.ldk + 64) * s.es());
    float *o = s.put<float>(nullptr, (size_t)xr * W.rows);
    void *dx = s.rows(x, n, k, xr, W.ldk);
    Pass p{&s.pm.nb, n, n > LG_MAXM, nullptr, nullptr, 0};
    if (w_up) gated(e, l, dx, W.ldk, p); else project(e, W, dx, W.ldk, p, o);
    const int ld = w_up ? l.down.ldk : W.rows;
    const std::vector<float> r = s.get(w_up ? s.pm.nb.act : (void *)o, (size_t)n * ld, !w_up || f32);
    for (int i = 0; i < n; i++) memcpy(out + (size_t)i * m, &r[(size_t)i * ld], (size_t)m * 4);
    s.pm.nb = PlanBuf();
    return 0;
}

extern "C" int lg_row_norm_host(float *x, int rows, int n, const float *add, const float *add_w, float mult, const float *norm_w, float eps,
                                int center, int f32, float *y) {
    if (rows < 1 || n < 1 || n > 16 * 1024 || (add && !add_w)) return -1;
    Scratch s(f32 != 0);
    LgRowNormArgs a{};
    a.x = s.put(x, (size_t)rows * n); a.ldx = a.n = n;
    if (add) { a.add = s.put(add, (size_t)rows * n); a.ld_add = n; a.add_w = s.put(add_w, n); }
    a.mult = mult; a.norm_w = s.put(norm_w, n); a.eps = eps; a.center = center;
    a.ldy = up(n, 64);
    a.y = s.put<uint8_t>(nullptr, (size_t)rows * a.ldy * s.es());
    launch_row_norm(&s.e, rows, a);
    const std::vector<float> r = s.get(a.y, (size_t)rows * a.ldy, f32 != 0);
    for (int i = 0; i < rows; i++) memcpy(y + (size_t)i * n, &r[(size_t)i * a.ldy], (size_t)n * 4);
    LG_CHECK(cudaMemcpy(x, a.x, (size_t)rows * n * 4, cudaMemcpyDeviceToHost));
    return 0;
}

// Attention over latent rows in the absorbed form: q [n][H][kv_rank + rot_dim], cache [pos + n][kv_rank + rot_dim] -> latent
// outputs [n][H][kv_rank].  form 0: the split kernel and its merge (bf16, n <= 8), 1: the row kernel.
extern "C" int lg_latent_attn_host(const float *q, const float *cache, const float *sink, int n, int H, int kv_rank, int rot_dim, int pos, int max_seq,
                                   float scale, int form, int f32, float *out) {
    if (n < 1 || H < 1 || kv_rank < 1 || rot_dim < 0 || pos < 0 || pos + n > max_seq || (form == 0 && (n > LG_MAXM || f32))) return -1;
    Scratch s(f32 != 0);
    Engine *e = &s.e;
    PlanLayer l;
    l.p = lg_plan_layer{};
    l.p.heads = H; l.p.kv_rank = kv_rank; l.p.rot_dim = rot_dim; l.p.scale = scale; l.p.dim = l.p.vdim = 16; l.p.ff = 0;
    layer_sizes(l);
    l.rt = l.kvp > 512 || lg_latent_dec_smem(1, l.ldc) > PLAN_SMEM_MAX ? 0 : lg_latent_dec_smem(2, l.ldc) <= PLAN_SMEM_MAX ? 2 : 1;
    if (form == 0 && !l.rt) return -2;
    auto padded = [&](const float *src, int rows) {            // [latent | 0 | key part | 0]
        std::vector<float> p((size_t)rows * l.ldc, 0.0f);
        for (int r = 0; r < rows; r++) {
            memcpy(&p[(size_t)r * l.ldc], src + (size_t)r * (kv_rank + rot_dim), (size_t)kv_rank * 4);
            memcpy(&p[(size_t)r * l.ldc + l.kvp], src + (size_t)r * (kv_rank + rot_dim) + kv_rank, (size_t)rot_dim * 4);
        }
        return p;
    };
    const int seq = cache_rows(max_seq);
    const std::vector<float> pq = padded(q, n * H), pc = padded(cache, pos + n);
    void *dq = s.rows(pq.data(), n * H, l.ldc, n * H, l.ldc), *dc = s.rows(pc.data(), pos + n, l.ldc, seq, l.ldc);
    int *dpos = s.put(&pos, 1);
    l.sink = s.put(sink, H);
    void *ol = s.put<uint8_t>(nullptr, (size_t)n * H * l.kvp * s.es());
    if (form == 1) {
        LgLatentRowsArgs ra{};
        ra.q = dq; ra.cache = dc; ra.ldc = l.ldc; ra.kvp = l.kvp; ra.H = H; ra.sink = l.sink; ra.scale = scale; ra.pos = dpos; ra.out = ol;
        launch_latent_rows(e, l, n, ra);
    } else {
        s.pm.seq_alloc = seq;
        s.pm.C = latent_splits(e, H, max_seq);
        s.pm.part = s.put<float>(nullptr, (size_t)n * H * l.kvp * s.pm.C);
        s.pm.part_ml = s.put<float2>(nullptr, (size_t)n * H * s.pm.C);
        launch_latent_dec(e, l, n, dq, dc, dpos, ol);
        s.pm.part = nullptr; s.pm.part_ml = nullptr;
    }
    const std::vector<float> r = s.get(ol, (size_t)n * H * l.kvp, f32 != 0);
    for (int i = 0; i < n * H; i++) memcpy(out + (size_t)i * kv_rank, &r[(size_t)i * l.kvp], (size_t)kv_rank * 4);
    return 0;
}

// The prompt block's attention: q [n][H][dim + rot_dim] (rotated), k [pos + n][H][dim], k_rot [pos + n][rot_dim],
// v [pos + n][H][vdim], gate [n][H][vdim] -> [n][H][vdim].
extern "C" int lg_latent_prompt_attn_host(const float *q, const float *k, const float *k_rot, const float *v, const float *gate, const float *sink,
                                          int n, int H, int dim, int rot_dim, int vdim, int pos, float scale, float *out) {
    if (n < 1 || H < 1 || dim < 1 || rot_dim < 1 || vdim < 1 || vdim > 256 || pos < 0) return -1;
    Scratch s(false);
    Engine *e = &s.e;
    PlanLayer l;
    l.p = lg_plan_layer{};
    l.p.heads = H; l.p.dim = dim; l.p.rot_dim = rot_dim; l.p.vdim = vdim; l.p.kv_rank = 16; l.p.scale = scale; l.p.ff = 0;
    layer_sizes(l);
    if (lg_latent_pf_smem(l.dimp, l.rotp, l.vdp) > PLAN_SMEM_MAX) return -2;
    const int keys = pos + n, seq = cache_rows(keys), cap = up(n, 128), qh = l.dimp + l.rotp, ldq = up(H * qh, 32), ldk = up(H * l.dimp, 32), ldo = up(H * l.vdp, 64);
    std::vector<float> hq((size_t)n * ldq), hk((size_t)keys * ldk), hc((size_t)keys * l.ldc), hv((size_t)H * l.vdp * seq), hg((size_t)n * H * l.vdp);
    for (int h = 0; h < H; h++) {
        for (int t = 0; t < n; t++) {
            memcpy(&hq[(size_t)t * ldq + h * qh], q + ((size_t)t * H + h) * (dim + rot_dim), (size_t)dim * 4);
            memcpy(&hq[(size_t)t * ldq + h * qh + l.dimp], q + ((size_t)t * H + h) * (dim + rot_dim) + dim, (size_t)rot_dim * 4);
            memcpy(&hg[((size_t)t * H + h) * l.vdp], gate + ((size_t)t * H + h) * vdim, (size_t)vdim * 4);
        }
        for (int t = 0; t < keys; t++) {
            memcpy(&hk[(size_t)t * ldk + h * l.dimp], k + ((size_t)t * H + h) * dim, (size_t)dim * 4);
            for (int j = 0; j < vdim; j++) hv[((size_t)h * l.vdp + j) * seq + t] = v[((size_t)t * H + h) * vdim + j];
        }
    }
    for (int t = 0; t < keys; t++) memcpy(&hc[(size_t)t * l.ldc + l.kvp], k_rot + (size_t)t * rot_dim, (size_t)rot_dim * 4);
    s.pm.seq_alloc = seq;
    l.uk.rows = ldk; l.uv.rows = up(H * l.vdp, 32);
    s.pm.kx = (bf16 *)s.rows(hk.data(), keys, ldk, seq, ldk);
    s.pm.vx = (bf16 *)s.rows(hv.data(), H * l.vdp, seq, l.uv.rows, seq);
    l.sink = s.put(sink, H);
    void *at = s.put<bf16>(nullptr, (size_t)cap * ldo);
    launch_latent_prompt(e, l, n, cap, s.rows(hq.data(), n, ldq, cap, ldq), ldq, s.rows(hc.data(), keys, l.ldc, seq, l.ldc), s.put(hg.data(), hg.size()), H * l.vdp,
                         s.put(&pos, 1), at, ldo);
    const std::vector<float> r = s.get(at, (size_t)n * ldo, false);
    for (int t = 0; t < n; t++)
        for (int h = 0; h < H; h++) memcpy(out + ((size_t)t * H + h) * vdim, &r[(size_t)t * ldo + h * l.vdp], (size_t)vdim * 4);
    s.pm.kx = s.pm.vx = nullptr;
    return 0;
}

// Input projections of a layer whose branches run side by side: out = w x [n][m], act = relu(w_up x_up)^2 [n][m_up].
extern "C" int lg_dense_pair_host(const float *w, int m, const float *w_up, int m_up, int k, const float *x, const float *x_up, int n, int f32,
                                  float *out, float *act) {
    if (m < 1 || m_up < 1 || k < 1 || n < 1) return -1;
    Scratch s(f32 != 0);
    Engine *e = &s.e;
    const int r0 = up(m, 32), r1 = up(m_up, 32), xr = up(n, 128), ld = up(k, 64);
    MatBuild b(e, r0 + r1, k);
    for (int r = 0; r < m; r++) for (int i = 0; i < k; i++) b.put((size_t)r * b.ldk + i, w[(size_t)r * k + i]);
    for (int r = 0; r < m_up; r++) for (int i = 0; i < k; i++) b.put((size_t)(r0 + r) * b.ldk + i, w_up[(size_t)r * k + i]);
    const DMat both = b.upload(e), a = rows_of(e, both, 0, r0), u = rows_of(e, both, r0, r1);
    s.mem.push_back(both.w);
    void *dx = s.rows(x, n, k, xr, ld), *du = s.rows(x_up, n, k, xr, ld);
    float *o = s.put<float>(nullptr, (size_t)xr * r0), *g = s.put<float>(nullptr, (size_t)xr * r1);
    void *ac = s.put<uint8_t>(nullptr, (size_t)xr * r1 * s.es());
    if (f32) {
        launch_f32(e, a, dx, ld, n, o, r0);
        launch_f32(e, u, du, ld, n, g, r1);
        launch_k(e, lg_dn_relu2_rows, dim3((r1 + 255) / 256, n), dim3(256), 0, (const float *)g, r1, r1, (float *)ac, r1);
    } else if (n > LG_MAXM) {
        launch_dn_gemm<DN_G_F32>(e, a, dx, ld, xr, n, o, r0);
        launch_dn_gemm<DN_G_RELU2>(e, u, du, ld, xr, n, ac, r1);
    } else {
        LgDnGemvArgs v{};
        v.x = (const bf16 *)dx; v.x2 = (const bf16 *)du; v.ldx = ld; v.M = n; v.split_tile = r0 / 16; v.out = o; v.ldo = r0; v.outh = (bf16 *)ac; v.ldoh = r1;
        launch_dn_gemv<DN_PAIR, false>(e, both, v);
    }
    const std::vector<float> ro = s.get(o, (size_t)n * r0, true), ra = s.get(ac, (size_t)n * r1, f32 != 0);
    for (int i = 0; i < n; i++) {
        memcpy(out + (size_t)i * m, &ro[(size_t)i * r0], (size_t)m * 4);
        memcpy(act + (size_t)i * m_up, &ra[(size_t)i * r1], (size_t)m_up * 4);
    }
    return 0;
}

// x += add + bias (either may be null), then the RMS norms of x with two weights.
extern "C" int lg_row_norm_pair_host(float *x, int rows, int n, const float *add, const float *bias, const float *norm_w, const float *norm_w2, float eps,
                                     int f32, float *y, float *y2) {
    if (rows < 1 || n < 1 || n > 16 * 1024 || !norm_w || !norm_w2) return -1;
    Scratch s(f32 != 0);
    LgRowNormArgs a{};
    a.x = s.put(x, (size_t)rows * n); a.ldx = a.n = n;
    if (add) { a.add = s.put(add, (size_t)rows * n); a.ld_add = n; }
    if (bias) a.bias = s.put(bias, n);
    a.norm_w = s.put(norm_w, n); a.norm_w2 = s.put(norm_w2, n); a.eps = eps; a.ldy = up(n, 64);
    a.y = s.put<uint8_t>(nullptr, (size_t)rows * a.ldy * s.es()); a.y2 = s.put<uint8_t>(nullptr, (size_t)rows * a.ldy * s.es());
    launch_row_norm_par(&s.e, rows, a);
    const std::vector<float> r = s.get(a.y, (size_t)rows * a.ldy, f32 != 0), r2 = s.get(a.y2, (size_t)rows * a.ldy, f32 != 0);
    for (int i = 0; i < rows; i++) {
        memcpy(y + (size_t)i * n, &r[(size_t)i * a.ldy], (size_t)n * 4);
        memcpy(y2 + (size_t)i * n, &r2[(size_t)i * a.ldy], (size_t)n * 4);
    }
    LG_CHECK(cudaMemcpy(x, a.x, (size_t)rows * n * 4, cudaMemcpyDeviceToHost));
    return 0;
}

// A mixer between its projections, block by block: rows [total][projected columns without padding] (grouped: q | k | v; state-space:
// z | x | B | C | step sizes) -> out [total][heads vdim], what the output product would read.  Block b runs tokens pos[b] .. pos[b] + m[b]
// (more than 8: as a prompt block), in the order given, so that positions can be run again.  w: grouped { q, k, v filters, lq1, lk1,
// lq2, lk2 }, state-space { filters, filter bias, dt_bias, A_log, D, norm weight }.  plain != 0: the kernels that hold every size.
extern "C" int lg_mixer_blocks_host(const struct lg_plan_layer *layer, float eps, int max_seq, const float *const *w, const float *rows, int total,
                                    const int *pos, const int *m, int n_blocks, int plain, int f32, float *out) {
    if (layer->mixer != LG_MIX_GROUPED && layer->mixer != LG_MIX_SSM) return -1;
    Scratch s(f32 != 0);
    Engine *e = &s.e;
    struct lg_plan plan{};
    struct lg_plan_layer pl = *layer;
    pl.ff = 0;
    plan.n_layer = 1; plan.width = 32; plan.vocab = 1; plan.layer = &pl; plan.form = LG_FORM_PARALLEL; plan.norm_eps = eps;
    s.pm.plan = &plan;
    s.pm.L.resize(1);
    PlanLayer &l = s.pm.L[0];
    l.p = pl; l.eps = eps;
    seq_layer_sizes(l);
    SeqWeights sw;
    auto take = [](const float *p, size_t n) { return std::vector<float>(p, p + n); };
    const int H = pl.heads, G = pl.kv_heads, M = pl.maps, inner = H * pl.vdim, gn = pl.groups * pl.state;
    const bool attn = pl.mixer == LG_MIX_GROUPED;
    if (attn) {
        const int ch[3] = {H * M * pl.dim, G * M * pl.dim, G * pl.vdim};
        for (int i = 0; i < 3; i++) sw.conv[i] = take(w[i], (size_t)ch[i] * pl.taps);
        if (M == 2) for (int i = 0; i < 4; i++) sw.lam[i] = take(w[3 + i], pl.dim);
    } else {
        sw.conv[0] = take(w[0], (size_t)(inner + 2 * gn) * pl.taps); sw.conv_b = take(w[1], inner + 2 * gn);
        sw.dt_bias = take(w[2], H); sw.a_log = take(w[3], H); sw.d = take(w[4], H); sw.norm = take(w[5], inner);
    }
    if (!seq_layer_weights(e, 0, l, sw)) { seq_layer_free(l); return -2; }
    if (plain) { l.chunked = 0; l.rt = 0; }
    l.act_off = up(l.at_cols, 64);
    l.in.rows = l.in_rows; l.in.ldk = 64; l.o.ldk = l.act_off;
    int cap = 128, bad = 0;
    for (int b = 0; b < n_blocks; b++) { cap = std::max(cap, up(m[b], 128)); bad |= m[b] < 1 || m[b] > PLAN_BLOCK || pos[b] < 0 || pos[b] + m[b] > std::min(total, max_seq); }
    if (bad) { seq_layer_free(l); return -1; }
    int kv_dim = 0, seq = 0, f16 = 0;
    void *k = nullptr, *v = nullptr;
    struct kvcache kv{};
    kv.n_layer = 1; kv.max_seq = max_seq; kv.kv_dim = &kv_dim; kv.seq = &seq; kv.f16 = &f16; kv.k = &k; kv.v = &v;
    seq_kv_init(&kv, &plan, f32 != 0);
    LG_CHECK(cudaDeviceSynchronize());
    s.pm.seq_alloc = up(max_seq, 128);
    seq_bind(e, &kv);
    e->x = nullptr;
    PlanBuf nb, wb;
    seq_buf_alloc(e, nb, LG_MAXM, true);
    seq_buf_alloc(e, wb, cap, false);
    // where unpadded column c of a projection row goes
    std::vector<int> at;
    auto sections = [&](int first, int n, int per, int to) { for (int i = 0; i < n; i++) for (int j = 0; j < per; j++) at.push_back(first + i * to + j); };
    if (attn) { sections(0, H * M, pl.dim, l.dimp); sections(l.q_cols, G * M, pl.dim, l.dimp); sections(l.q_cols + l.k_cols, G, pl.vdim, l.vdp); }
    else { sections(0, H, pl.vdim, l.vdp); sections(l.ch0, H, pl.vdim, l.vdp); sections(l.ch0 + H * l.vdp, 2 * pl.groups, pl.state, l.np); sections(l.dt_off, 1, H, H); }
    const int cols = (int)at.size();
    int *d_pos = s.put<int>(nullptr, 1);
    for (int b = 0; b < n_blocks; b++) {
        const bool wide = m[b] > LG_MAXM;
        PlanBuf &pb = wide ? wb : nb;
        std::vector<float> pad((size_t)m[b] * l.in_rows, 0.0f), dt((size_t)m[b] * std::max(1, l.in_rows - l.dt_off), 0.0f);
        for (int t = 0; t < m[b]; t++)
            for (int c = 0; c < cols; c++) {
                const float x = rows[(size_t)(pos[b] + t) * cols + c];
                pad[(size_t)t * l.in_rows + at[c]] = x;
                if (at[c] >= l.dt_off) dt[(size_t)t * (l.in_rows - l.dt_off) + at[c] - l.dt_off] = x;
            }
        if (wide && !f32) {
            std::vector<uint16_t> h(pad.size());
            for (size_t i = 0; i < pad.size(); i++) h[i] = bf16_bits(pad[i]);
            h2d_sync(pb.pj, h.data(), h.size() * 2);
            if (!attn) h2d_sync(pb.dt, dt.data(), dt.size() * 4);
        } else h2d_sync(pb.pj, pad.data(), pad.size() * 4);
        h2d_sync(d_pos, &pos[b], 4);
        Pass p{&pb, m[b], wide, nullptr, d_pos, pos[b]};
        launch_k(e, lg_seq_begin_kernel, dim3(1), dim3(32), 0, seq_ctl(&kv), (const int *)d_pos, m[b], wide ? 1 : 0, e->err);
        seq_mixer(e, &kv, l, 0, p, C_ALL);
        const std::vector<float> r = s.get(pb.at, (size_t)m[b] * l.o.ldk, f32 != 0);
        for (int t = 0; t < m[b]; t++)
            for (int h = 0; h < H; h++)
                memcpy(out + ((size_t)(pos[b] + t) * H + h) * pl.vdim, &r[(size_t)t * l.o.ldk + h * l.vdp], (size_t)pl.vdim * 4);
    }
    seq_layer_free(l);
    buf_free(nb, true); buf_free(wb, false);
    cudaFree(k); cudaFree(v); cudaFree(s.pm.part); cudaFree(s.pm.part_ml);
    s.pm.part = nullptr; s.pm.part_ml = nullptr; s.pm.plan = nullptr;
    return 0;
}
