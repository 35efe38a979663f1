// lg_plan_seq.cuh -- host side of the layers that add a mixer and a feed-forward side by side (lg_plan.cu includes it): grouped
// windowed attention and state-space mixers, their weights, sequence state and launches.
//
// Such a layer is two stacked input projections (one launch in a decode step), the mixer, and ONE output product over the mixer's
// and the feed-forward's rows side by side: W_o y + W_down act = [W_o | W_down] [y | act].

// ------------------------------------------------------------------------------------------
// loading
// ------------------------------------------------------------------------------------------
float *vec_offset(Engine *e, int L, const char *leaf, int n, float offset) {
    std::vector<float> f = row_f32(need(e, L, leaf, n, 0), 0);
    for (auto &x : f) x += offset;
    return upload_f32(f.data(), f.size());
}
// `sections` of `per` values of a vector, each padded to `to`
void put_sections(std::vector<float> &dst, size_t at, const std::vector<float> &src, size_t from, int sections, int per, int to) {
    for (int s = 0; s < sections; s++)
        for (int i = 0; i < per; i++) dst[at + (size_t)s * to + i] = src[from + (size_t)s * per + i];
}
// filters [channels][taps], channels from .. in padded sections, as [taps][nch]
void put_taps(std::vector<float> &dst, int nch, int at, const std::vector<float> &f, int from, int sections, int per, int to, int taps) {
    for (int s = 0; s < sections; s++)
        for (int i = 0; i < per; i++)
            for (int j = 0; j < taps; j++) dst[(size_t)j * nch + at + s * to + i] = f[(size_t)(from + s * per + i) * taps + j];
}
std::vector<float> mat_f32(const struct gguf_tensor *t) {
    std::vector<float> f;
    for (int r = 0; r < (int)t->dims[1]; r++) { const std::vector<float> row = row_f32(t, r); f.insert(f.end(), row.begin(), row.end()); }
    return f;
}
// rows [row0, row0 + rows) of a matrix as a matrix of its own
DMat rows_of(const Engine *e, const DMat &m, int row0, int rows) {
    DMat v = m;
    const size_t es = e->f32 ? 4 : 2;
    v.w = (uint8_t *)m.w + (size_t)row0 * m.ldk * es;
    v.rows = rows; v.rows_alloc = std::min(up(rows, 256), m.rows_alloc - row0);
    if (!e->f32)
        for (int i = 0; i < 2; i++) v.map[i] = tiled_map(v.w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, v.ldk, v.rows_alloc, (long long)v.ldk * 2, DN_GEMM_BK, 128 << i);
    return v;
}

// sizes of a layer that follow from the plan alone; the cache layout depends on them
void seq_layer_sizes(PlanLayer &l) {
    const struct lg_plan_layer &p = l.p;
    l.vdp = up(p.vdim, 16); l.ffp = up(p.ff, 16);
    l.mask = 31;
    while (l.mask + 1 < 16 + p.taps) l.mask = 2 * l.mask + 1;
    if (p.mixer == LG_MIX_GROUPED) {
        l.dimp = up(p.dim, 16);
        l.ch0 = 0;
        l.q_cols = p.heads * p.maps * l.dimp; l.k_cols = p.kv_heads * p.maps * l.dimp;
        l.nch = l.q_cols + l.k_cols + p.kv_heads * l.vdp;
        l.ldc = l.nch - l.q_cols;
        l.dt_off = l.nch;
        l.in_rows = up(l.nch, 32);
    } else {
        l.np = up(p.state, 16);
        l.npl = p.state <= 32 ? 1 : p.state <= 64 ? 2 : p.state <= 128 ? 4 : p.state <= 256 ? 8 : 0;
        l.nst = 32 * l.npl;
        l.ch0 = p.heads * l.vdp;
        l.nch = p.heads * l.vdp + 2 * p.groups * l.np;
        l.ldc = 0;
        l.dt_off = up(l.ch0 + l.nch, 32);
        l.in_rows = up(l.dt_off + p.heads, 32);
    }
    l.at_cols = p.heads * l.vdp;
}
// A slot's state block: [control | ring of projected rows | ring of raw step sizes | states]
struct SeqBlock { size_t ring, dt, state, bytes; };
SeqBlock seq_block(const PlanLayer &l, bool f32) {
    auto r = [](size_t n) { return (n + 255) / 256 * 256; };
    SeqBlock b;
    b.ring = 256;
    b.dt = b.ring + r((size_t)(l.mask + 1) * l.nch * (f32 ? 4 : 2));
    b.state = b.dt + (l.p.mixer == LG_MIX_SSM ? r((size_t)(l.mask + 1) * l.p.heads * 4) : 0);
    b.bytes = b.state + (l.p.mixer == LG_MIX_SSM ? r((size_t)l.p.heads * l.vdp * l.nst * 4) : 0);
    return b;
}
// cache rows of a slot: a windowed layer keeps a ring that holds the window and a wide block, in whole key tiles
int seq_rows(const PlanLayer &l, int max_seq) {
    const int all = up(max_seq, 128);
    return l.p.window > 0 ? (int)std::min<long long>(all, ((long long)l.p.window + PLAN_BLOCK + 64 + 127) / 128 * 128) : all;
}

// What a mixer holds besides its projections: filters [channels][taps] (of q, k, v, or of x | B | C), and the vectors of its kind.
struct SeqWeights { std::vector<float> conv[3], conv_b, dt_bias, a_log, d, norm, lam[4]; };

// false, after a message: sizes beyond what the kernels hold
bool seq_layer_weights(const Engine *e, int i, PlanLayer &l, const SeqWeights &w) {
    const struct lg_plan_layer &p = l.p;
    const int H = p.heads, G = p.kv_heads, M = p.maps;
    std::vector<float> cw((size_t)p.taps * l.nch, 0.0f);
    bool ok = true;
    if (p.mixer == LG_MIX_GROUPED) {
        put_taps(cw, l.nch, 0, w.conv[0], 0, H * M, p.dim, l.dimp, p.taps);
        put_taps(cw, l.nch, l.q_cols, w.conv[1], 0, G * M, p.dim, l.dimp, p.taps);
        put_taps(cw, l.nch, l.q_cols + l.k_cols, w.conv[2], 0, G, p.vdim, l.vdp, p.taps);
        l.out_mult = 1.0f;
        if (M == 2) {                        // weight of the second map
            double s[2] = {0.0, 0.0};
            for (int j = 0; j < 2; j++) for (int d = 0; d < p.dim; d++) s[j] += (double)w.lam[2 * j][d] * w.lam[2 * j + 1][d];
            l.lambda = (float)(exp(s[0]) - exp(s[1]) + (double)p.diff);
            l.out_mult = 1.0f - p.diff;
        }
        if (l.vdp > (M == 1 ? 256 : 128) || lg_win_pf_smem(M, l.dimp, l.vdp) > PLAN_SMEM_SMALL) l.chunked = 0;
        l.rt = !e->f32 && l.vdp <= 256 && lg_win_dec_smem(M, l.dimp, l.vdp) <= PLAN_SMEM_MAX;
        ok = (size_t)(M * (l.dimp + l.vdp) + M * 128) * 4 <= PLAN_SMEM_SMALL;
    } else {
        const int inner = H * p.vdim, gn = p.groups * p.state, part_n = inner / p.norm_groups;
        const int part[3][5] = {{0, 0, H, p.vdim, l.vdp}, {H * l.vdp, inner, p.groups, p.state, l.np}, {H * l.vdp + p.groups * l.np, inner + gn, p.groups, p.state, l.np}};
        std::vector<float> cb(l.nch, 0.0f), gn_w((size_t)H * l.vdp, 0.0f);
        for (auto &q : part) {                                             // x, B, C
            put_taps(cw, l.nch, q[0], w.conv[0], q[1], q[2], q[3], q[4], p.taps);
            put_sections(cb, q[0], w.conv_b, q[1], q[2], q[3], q[4]);
        }
        put_sections(gn_w, 0, w.norm, 0, H, p.vdim, l.vdp);
        l.conv_b = upload_f32(cb.data(), cb.size());
        l.dt_bias = upload_f32(w.dt_bias.data(), H); l.a_log = upload_f32(w.a_log.data(), H); l.d = upload_f32(w.d.data(), H);
        l.gnorm = upload_f32(gn_w.data(), gn_w.size());
        ok = l.npl && part_n <= (p.vdim % 4 || part_n % 4 ? 16 : 32) * 1024;
        l.vs = std::min(l.vdp, 64);
        if (l.np > 256) l.chunked = 0;
    }
    l.conv_w = upload_f32(cw.data(), cw.size());
    if (!ok) fprintf(stderr, "lg_b200: layer %d: sizes beyond what the kernels hold\n", i);
    return ok;
}

void seq_layer_load(Engine *e, int i, PlanLayer &l) {
    PlanModel *pm = e->plan;
    const struct lg_plan *P = pm->plan;
    const struct lg_plan_layer &p = l.p;
    const int W = P->width, H = p.heads, G = p.kv_heads, M = p.maps;
    SeqWeights w;
    MatBuild b(e, l.in_rows + (p.ff ? up(l.ffp, 32) : 0), W);
    if (p.mixer == LG_MIX_GROUPED) {
        put_groups(b, 0, need(e, i, "attn_q", H * M * p.dim, W), H * M, p.dim, l.dimp);
        put_groups(b, l.q_cols, need(e, i, "attn_k", G * M * p.dim, W), G * M, p.dim, l.dimp);
        put_groups(b, l.q_cols + l.k_cols, need(e, i, "attn_v", G * p.vdim, W), G, p.vdim, l.vdp);
        w.conv[0] = mat_f32(need(e, i, "attn_q_conv", H * M * p.dim, p.taps));
        w.conv[1] = mat_f32(need(e, i, "attn_k_conv", G * M * p.dim, p.taps));
        w.conv[2] = mat_f32(need(e, i, "attn_v_conv", G * p.vdim, p.taps));
        static const char *const names[4] = {"attn_lambda_q1", "attn_lambda_k1", "attn_lambda_q2", "attn_lambda_k2"};
        if (M == 2) for (int j = 0; j < 4; j++) w.lam[j] = row_f32(need(e, i, names[j], p.dim, 0), 0);
    } else {
        const int inner = H * p.vdim, gn = p.groups * p.state;
        const struct gguf_tensor *t = need(e, i, "ssm_in", 2 * inner + 2 * gn + H, W);
        auto sections = [&](int dst, int src, int n, int per, int to) {
            for (int s = 0; s < n; s++) for (int r = 0; r < per; r++) b.row(dst + s * to + r, t, src + s * per + r);
        };
        sections(0, 0, H, p.vdim, l.vdp);                                  // z, x, B, C, step sizes
        sections(l.ch0, inner, H, p.vdim, l.vdp);
        sections(l.ch0 + H * l.vdp, 2 * inner, 2 * p.groups, p.state, l.np);
        sections(l.dt_off, 2 * inner + 2 * gn, 1, H, H);
        w.conv[0] = mat_f32(need(e, i, "ssm_conv1d", inner + 2 * gn, p.taps));
        w.conv_b = row_f32(need(e, i, "ssm_conv1d_bias", inner + 2 * gn, 0), 0);
        w.dt_bias = row_f32(need(e, i, "ssm_dt_bias", H, 0), 0); w.a_log = row_f32(need(e, i, "ssm_a_log", H, 0), 0); w.d = row_f32(need(e, i, "ssm_d", H, 0), 0);
        w.norm = row_f32(need(e, i, "ssm_norm", inner, 0), 0);
    }
    if (!seq_layer_weights(e, i, l, w)) exit(1);
    const struct gguf_tensor *o = need(e, i, "attn_output", W, H * p.vdim);
    l.act_off = up(l.at_cols, 64);
    MatBuild c(e, W, l.act_off + (p.ff ? up(l.ffp, 64) : 0));
    for (int r = 0; r < W; r++) c.row(r, o, r, p.vdim, l.vdp);
    if (p.ff) {
        const struct gguf_tensor *u = need(e, i, "ffn_up", p.ff, W), *d = need(e, i, "ffn_down", W, p.ff);
        for (int r = 0; r < p.ff; r++) b.row(l.in_rows + r, u, r);
        for (int r = 0; r < W; r++) c.row(r, d, r, 0, 0, l.act_off);
        l.norm2 = vec_offset(e, i, "ffn_norm", W, P->norm_offset);
    }
    l.inup = b.upload(e);
    l.in = rows_of(e, l.inup, 0, l.in_rows);
    if (p.ff) l.gu = rows_of(e, l.inup, l.in_rows, up(l.ffp, 32));
    l.o = c.upload(e);
    l.norm1 = vec_offset(e, i, "attn_norm", W, P->norm_offset);
}
void seq_layer_free(PlanLayer &l) {
    for (float *v : {l.conv_w, l.conv_b, l.dt_bias, l.a_log, l.d, l.gnorm}) cudaFree(v);
}
// The kernels of a decode step ask for one division of an SM's memory between cache and shared memory (percent of the latter): where it
// changes from one kernel to the next, the SM has to run empty first, and nothing overlaps.  64 KB hold the mixers' CTAs and leave the
// weight stream of the matmuls the cache lines its loads in flight need.
constexpr int STEP_CARVEOUT = 28;
template <typename K> void same_carveout(K kernel) { LG_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, STEP_CARVEOUT)); }
template <int EPI> void gemv_carveout() {
    same_carveout(lg_dn_gemv_kernel<EPI, 1, false>); same_carveout(lg_dn_gemv_kernel<EPI, 2, false>);
    same_carveout(lg_dn_gemv_kernel<EPI, 4, false>); same_carveout(lg_dn_gemv_kernel<EPI, 8, false>);
}
template <typename T> void step_carveout() {
    same_carveout(lg_ssm_step_kernel<T, 1, false>); same_carveout(lg_ssm_step_kernel<T, 2, false>);
    same_carveout(lg_ssm_step_kernel<T, 4, false>); same_carveout(lg_ssm_step_kernel<T, 8, false>);
}
constexpr size_t SSM_SMEM = lg_ssm_step_smem(LG_CONV_MAX_TAPS, 256);
void seq_attributes() {
    smem_attr(lg_dn_gemm_kernel<128, DN_G_RELU2>, dn_gemm_smem<128>()); smem_attr(lg_dn_gemm_kernel<256, DN_G_RELU2>, dn_gemm_smem<256>());
    smem_attr(lg_ssm_step_kernel<float, 1, false>, SSM_SMEM); smem_attr(lg_ssm_step_kernel<float, 2, false>, SSM_SMEM);
    smem_attr(lg_ssm_step_kernel<float, 4, false>, SSM_SMEM); smem_attr(lg_ssm_step_kernel<float, 8, false>, SSM_SMEM);
    smem_attr(lg_ssm_step_kernel<bf16, 1, false>, SSM_SMEM); smem_attr(lg_ssm_step_kernel<bf16, 2, false>, SSM_SMEM);
    smem_attr(lg_ssm_step_kernel<bf16, 4, false>, SSM_SMEM); smem_attr(lg_ssm_step_kernel<bf16, 8, false>, SSM_SMEM);
    gemv_carveout<DN_STORE>(); gemv_carveout<DN_PAIR>(); gemv_carveout<DN_HEAD>();
    step_carveout<bf16>();
    same_carveout(lg_row_norm_kernel<bf16, 2, 4, true>); same_carveout(lg_row_norm_kernel<bf16, 4, 4, true>); same_carveout(lg_row_norm_kernel<bf16, 16, 1, true>);
    same_carveout(lg_conv_kernel<float, bf16, 2>); same_carveout(lg_conv_kernel<float, bf16, 3>); same_carveout(lg_conv_kernel<float, bf16, 4>);
    same_carveout(lg_conv_any_kernel<float, bf16>);
    same_carveout(lg_gated_norm_kernel<float, bf16, 4, 2>); same_carveout(lg_gated_norm_kernel<float, bf16, 4, 8>);
    same_carveout(lg_gated_norm_kernel<float, bf16, 1, 4>); same_carveout(lg_gated_norm_kernel<float, bf16, 1, 16>);
    same_carveout(lg_win_dec_attn_kernel<1, 4>); same_carveout(lg_win_dec_attn_kernel<2, 4>); same_carveout(lg_win_dec_attn_kernel<2, 8>);
    same_carveout(lg_win_merge_kernel<1>); same_carveout(lg_win_merge_kernel<2>);
    same_carveout(lg_dn_embed_rows<bf16>); same_carveout(lg_seq_begin_kernel);
    smem_attr(lg_ssd_state_kernel, PLAN_SMEM_MAX - 2048); smem_attr(lg_ssd_out_kernel, PLAN_SMEM_MAX - 2048);
    smem_attr(lg_win_dec_attn_kernel<1, 4>); smem_attr(lg_win_dec_attn_kernel<2, 4>); smem_attr(lg_win_dec_attn_kernel<2, 8>);
    smem_attr(lg_win_pf_attn_kernel<1>, PLAN_SMEM_SMALL); smem_attr(lg_win_pf_attn_kernel<2>, PLAN_SMEM_SMALL);
    smem_attr(lg_win_attn_rows_kernel<float, 1>, PLAN_SMEM_SMALL); smem_attr(lg_win_attn_rows_kernel<float, 2>, PLAN_SMEM_SMALL);
    smem_attr(lg_win_attn_rows_kernel<bf16, 1>, PLAN_SMEM_SMALL); smem_attr(lg_win_attn_rows_kernel<bf16, 2>, PLAN_SMEM_SMALL);
}

void seq_buf_alloc(Engine *e, PlanBuf &b, int cap, bool narrow) {
    PlanModel *pm = e->plan;
    const int W = pm->plan->width;
    const size_t es = e->f32 ? 4 : 2;
    const bool f32_rows = narrow || e->f32;                      // projection rows: f32, or bf16 with the step sizes in f32 of their own
    size_t pj = 0, o = up(W, 32), gu = 0, q = 16, at = 0, cv = 16, y = 16, heads = 0, ds = 0, chunks = (size_t)(cap + LG_SSD_Q - 1) / LG_SSD_Q;
    for (auto &l : pm->L) {
        pj = std::max(pj, (size_t)l.in.rows); at = std::max(at, (size_t)l.o.ldk);
        if (l.p.ff) gu = std::max(gu, (size_t)l.gu.rows);
        if (l.p.mixer == LG_MIX_GROUPED) q = std::max(q, (size_t)l.q_cols);
        else {
            cv = std::max(cv, (size_t)l.nch); y = std::max(y, (size_t)l.at_cols); heads = std::max(heads, (size_t)l.p.heads);
            if (l.chunked) ds = std::max(ds, (size_t)l.p.heads * l.np * l.vdp);
        }
    }
    auto bytes = [&](size_t per, size_t el) { return (void *)dalloc<uint8_t>(((size_t)cap * per + 256) * el); };
    b.cap = cap;
    b.x = narrow ? e->x : dalloc<float>((size_t)cap * W);
    b.pj = (float *)bytes(pj, f32_rows ? 4 : 2);
    b.o = dalloc<float>(cap * o);
    if (e->f32) b.gu = dalloc<float>(cap * gu + 16);
    b.h = bytes(up(W, 64), es); b.h2 = bytes(up(W, 64), es); b.q = bytes(q, es); b.at = bytes(at, es);
    b.y = bytes(y, narrow ? 4 : es);
    if (!narrow) {
        b.cv = bytes(cv, es);
        b.pos = dalloc<int>(1);
        if (!e->f32) {
            b.dt = dalloc<float>((size_t)cap * up((int)heads, 32) + 16);
            b.s_hi = dalloc<bf16>(chunks * ds + 16); b.s_lo = dalloc<bf16>(chunks * ds + 16);
        }
    }
}

// ------------------------------------------------------------------------------------------
// cache and sequence state
// ------------------------------------------------------------------------------------------
LgSeqCtl *seq_ctl(const struct kvcache *kv) { return (LgSeqCtl *)kv->v[0]; }     // at the head of the first slot's state block

// Whether a block may start at pos: it starts a sequence, or the states reach there.  n: tokens of the block the caller is about to run
// (they leave states for every position of a narrow block, behind a wide one), n < 0: rounds on the device that the host does not follow.
bool plan_start(Engine *e, const struct kvcache *kv, int pos, int n, bool wide) {
    PlanModel *pm = e->plan;
    if (pm->plan->form != LG_FORM_PARALLEL) return true;
    if (pos != 0 && (pm->st_lo < 0 || pm->st_kv != kv || pos < pm->st_lo || pos > pm->st_hi)) {
        LgSeqCtl c;                                              // the host has lost track: ask the device
        LG_CHECK(cudaMemcpyAsync(&c, seq_ctl(kv), sizeof c, cudaMemcpyDeviceToHost, e->stream));
        LG_CHECK(cudaStreamSynchronize(e->stream));
        if (pos < c.base || pos > c.base + c.have) return false;
    }
    pm->st_kv = kv;
    if (n < 0) pm->st_lo = -1;
    else { pm->st_lo = wide ? pos + n : pos; pm->st_hi = pos + n; }
    return true;
}
// the rows or states behind a saved prefix of n tokens
bool plan_prefix(struct kvcache *kv, int n, bool restore, cudaStream_t s) {
    (void)n;
    for (int L = 0; L < kv->n_layer; L++) {
        if (!kv->v[L]) continue;
        size_t bytes = 0;
        LG_CHECK(cudaMemcpy(&bytes, (uint8_t *)kv->v[L] + 128, sizeof bytes, cudaMemcpyDeviceToHost));
        if (!restore) {
            LG_CHECK(cudaMalloc(&kv->px_v[L], bytes));
            LG_CHECK(cudaMemcpy(kv->px_v[L], kv->v[L], bytes, cudaMemcpyDeviceToDevice));
        } else if (kv->px_v[L]) LG_CHECK(cudaMemcpyAsync(kv->v[L], kv->px_v[L], bytes, cudaMemcpyDeviceToDevice, s));
    }
    return true;
}
int seq_kv_init(struct kvcache *kv, const struct lg_plan *P, bool f32) {
    for (int r = 0; r < kv->n_layer; r++) {
        PlanLayer l;
        l.p = P->layer[lg_plan_run_layer(P, r, nullptr)];
        seq_layer_sizes(l);
        kv->kv_dim[r] = l.ldc;
        kv->f16[r] = f32 ? 0 : 2;
        if (l.ldc) {
            kv->seq[r] = seq_rows(l, kv->max_seq);
            const size_t bytes = (size_t)kv->seq[r] * l.ldc * (f32 ? 4 : 2);
            LG_CHECK(cudaMalloc(&kv->k[r], bytes));
            LG_CHECK(cudaMemset(kv->k[r], 0, bytes));
        }
        const size_t bytes = seq_block(l, f32).bytes;
        LG_CHECK(cudaMalloc(&kv->v[r], bytes));
        LG_CHECK(cudaMemset(kv->v[r], 0, bytes));
        LG_CHECK(cudaMemcpy((uint8_t *)kv->v[r] + 128, &bytes, sizeof bytes, cudaMemcpyHostToDevice));       // the block's own size
    }
    return 0;
}
int win_splits(const Engine *e, const PlanLayer &l, int max_seq) {
    const int tiles = l.p.window > 0 ? std::min(up(max_seq, LG_WD_S) / LG_WD_S, (l.p.window + LG_MAXM + 62) / LG_WD_S + 1) : up(max_seq, LG_WD_S) / LG_WD_S;
    return std::max(1, std::min({e->sm_count / l.p.kv_heads, tiles, LG_WM_MAXC}));
}
void seq_bind(Engine *e, const struct kvcache *kv) {
    PlanModel *pm = e->plan;
    size_t part = 0, ml = 0;
    for (auto &l : pm->L) {
        if (l.p.mixer != LG_MIX_GROUPED || !l.rt) continue;
        l.C = win_splits(e, l, kv->max_seq);
        ml = std::max(ml, (size_t)l.C * LG_MAXM * l.p.heads * l.p.maps);
        part = std::max(part, (size_t)l.C * LG_MAXM * l.p.heads * l.p.maps * l.vdp);
    }
    if (ml) { pm->part = dalloc<float>(part); pm->part_ml = dalloc<float2>(ml); }
    pm->st_lo = -1;
}

// ------------------------------------------------------------------------------------------
// mixers
// ------------------------------------------------------------------------------------------
template <typename TI, typename T> void conv_go(Engine *e, LgConvArgs a) {
    a.run = a.taps >= 2 && a.taps <= 4 ? LG_CONV_RUN : std::max(16, a.taps - 1);          // the first run alone reads the ring
    const dim3 grid((a.nch / LG_CONV_V + LG_CONV_THREADS - 1) / LG_CONV_THREADS, (a.M + a.run - 1) / a.run), block(LG_CONV_THREADS);
    switch (a.taps) {
    case 2: launch_k(e, lg_conv_kernel<TI, T, 2>, grid, block, 0, a); break;
    case 3: launch_k(e, lg_conv_kernel<TI, T, 3>, grid, block, 0, a); break;
    case 4: launch_k(e, lg_conv_kernel<TI, T, 4>, grid, block, 0, a); break;
    default: launch_k(e, lg_conv_any_kernel<TI, T>, grid, block, 0, a); break;
    }
}
void launch_conv(Engine *e, const LgConvArgs &a, bool f32_src) {
    if (e->f32) conv_go<float, float>(e, a);
    else if (f32_src) conv_go<float, bf16>(e, a);
    else conv_go<bf16, bf16>(e, a);
}
template <typename T, bool WIDE> void step_go(Engine *e, const PlanLayer &l, const LgSsmStepArgs &a) {
    const dim3 grid(l.p.heads, l.vdp / LG_SSM_ROWS), block(LG_SSM_THREADS);
    const size_t sm = WIDE ? 0 : lg_ssm_step_smem(a.taps, a.np);
    switch (l.npl) {
    case 1: launch_k(e, lg_ssm_step_kernel<T, 1, WIDE>, grid, block, sm, a); break;
    case 2: launch_k(e, lg_ssm_step_kernel<T, 2, WIDE>, grid, block, sm, a); break;
    case 4: launch_k(e, lg_ssm_step_kernel<T, 4, WIDE>, grid, block, sm, a); break;
    default: launch_k(e, lg_ssm_step_kernel<T, 8, WIDE>, grid, block, sm, a); break;
    }
}
void launch_ssm_step(Engine *e, const PlanLayer &l, const LgSsmStepArgs &a, bool wide) {
    if (e->f32) { if (wide) step_go<float, true>(e, l, a); else step_go<float, false>(e, l, a); }
    else if (wide) step_go<bf16, true>(e, l, a);
    else step_go<bf16, false>(e, l, a);
}
// a block's convolved rows u [n][x | B | C] -> y, the state advanced in place
void launch_ssd(Engine *e, const PlanLayer &l, int n, int cap, const void *u, const float *dt, int ld_dt, const PlanBuf &b, float *state, bool fresh, void *y, int ldy) {
    PlanModel *pm = e->plan;
    const int chunks = (n + LG_SSD_Q - 1) / LG_SSD_Q, H = l.p.heads, all = (cap + LG_SSD_Q - 1) / LG_SSD_Q * H * l.np;
    LgSsdArgs a{};
    a.dt = dt; a.ld_dt = ld_dt; a.dt_bias = l.dt_bias; a.a_log = l.a_log; a.d = l.d;
    a.heads = H; a.groups = l.p.groups; a.np = l.np; a.vdp = l.vdp; a.vs = l.vs; a.n = n;
    a.nst = l.nst; a.chunks = chunks; a.fresh = fresh; a.state = state; a.hi = b.s_hi; a.lo = b.s_lo; a.y = (bf16 *)y; a.ldy = ldy; a.err = e->err;
    const CUtensorMap &mu = buf_map(pm, u, l.nch, l.nch, cap, LG_SSD_Q);
    LgSsdArgs c = a;
    const int tiles = H * ((l.np + 127) / 128);
    c.vs = std::min(l.vdp, 64);                                  // fewer value columns per CTA while there are SMs without one
    while (c.vs > 16 && tiles * ((l.vdp + c.vs - 1) / c.vs) * 2 <= e->sm_count + e->sm_count / 8) c.vs = up(c.vs / 2, 16);
    launch_k(e, lg_ssd_state_kernel, dim3(H, (l.vdp + c.vs - 1) / c.vs, (l.np + 127) / 128), dim3(LG_SSD_STATE_THREADS), lg_ssd_state_smem(c.vs), mu, c);
    // heads of a group that one CTA takes in turn (they share C B^T): the fewest rounds of CTAs, at about three heads' time to start one
    const int per = H / l.p.groups, slices = (l.vdp + l.vs - 1) / l.vs;
    long long best = 0;
    for (int sp = 1; sp <= per; sp++) {
        const long long rounds = ((long long)chunks * l.p.groups * slices * sp + e->sm_count - 1) / e->sm_count, cost = rounds * ((per + sp - 1) / sp + 3);
        if (!best || cost < best) { best = cost; a.splits = sp; }
    }
    a.stages = lg_ssd_out_smem(l.np, 2) <= PLAN_SMEM_MAX - 2048 ? 2 : 1;
    const dim3 grid(chunks, l.p.groups * a.splits, slices);
    launch_k(e, lg_ssd_out_kernel, grid, dim3(LG_SSD_OUT_THREADS), lg_ssd_out_smem(l.np, a.stages), mu,
             buf_map(pm, b.s_hi, l.vdp, l.vdp, all, l.np), buf_map(pm, b.s_lo, l.vdp, l.vdp, all, l.np), a);
}
template <typename TI, typename TO> void gated_norm_go(Engine *e, int n, int parts, const LgGatedNormArgs &a) {
    const bool v4 = a.n % 4 == 0 && a.vd % 4 == 0;
    if (v4 && a.n <= 1024 && n > LG_MAXM) {           // (few rows: more threads per part)
        const dim3 grid((n * parts + LG_GN_WARPS - 1) / LG_GN_WARPS), block(LG_GN_WARPS * 32);
        if (a.n <= 512) launch_k(e, lg_gated_norm_warp_kernel<TI, TO, 4>, grid, block, 0, a, parts, n);
        else launch_k(e, lg_gated_norm_warp_kernel<TI, TO, 8>, grid, block, 0, a, parts, n);
        return;
    }
    const int items = v4 ? a.n / 4 : a.n, ipt_few = v4 ? 2 : 4;
    const int threads = std::min(1024, std::max(32, up((items + ipt_few - 1) / ipt_few, 32)));
    const bool few = (items + threads - 1) / threads <= ipt_few;
    const dim3 grid(parts, n), block(threads);
    if (v4) { if (few) launch_k(e, lg_gated_norm_kernel<TI, TO, 4, 2>, grid, block, 0, a); else launch_k(e, lg_gated_norm_kernel<TI, TO, 4, 8>, grid, block, 0, a); }
    else if (few) launch_k(e, lg_gated_norm_kernel<TI, TO, 1, 4>, grid, block, 0, a);
    else launch_k(e, lg_gated_norm_kernel<TI, TO, 1, 16>, grid, block, 0, a);
}
void launch_gated_norm(Engine *e, int n, int parts, const LgGatedNormArgs &a, bool f32_rows) {
    if (e->f32) gated_norm_go<float, float>(e, n, parts, a);
    else if (f32_rows) gated_norm_go<float, bf16>(e, n, parts, a);
    else gated_norm_go<bf16, bf16>(e, n, parts, a);
}
// grouped attention of n tokens at *pos over the cache; form 0: split + merge (n <= LG_MAXM), 1: rows, 2: prompt block
void launch_win(Engine *e, const PlanLayer &l, int form, int n, int q_rows, LgWinArgs a) {
    PlanModel *pm = e->plan;
    const struct lg_plan_layer &p = l.p;
    a.H = p.heads; a.G = p.kv_heads; a.dimp = l.dimp; a.vd = p.vdim; a.vdp = l.vdp; a.window = p.window; a.ldc = l.ldc; a.v_off = l.k_cols;
    a.ldq = l.q_cols; a.scale = p.scale; a.lambda = l.lambda; a.out_mult = l.out_mult; a.eps = l.eps; a.n = n; a.part = pm->part; a.part_ml = pm->part_ml; a.err = e->err;
    const bool two = p.maps == 2;
    if (form == 1) {
        const size_t sm = (size_t)(p.maps * (l.dimp + l.vdp) + p.maps * 128) * 4;
        const dim3 grid(p.heads, n), block(128);
        if (e->f32) { if (two) launch_k(e, lg_win_attn_rows_kernel<float, 2>, grid, block, sm, a); else launch_k(e, lg_win_attn_rows_kernel<float, 1>, grid, block, sm, a); }
        else if (two) launch_k(e, lg_win_attn_rows_kernel<bf16, 2>, grid, block, sm, a);
        else launch_k(e, lg_win_attn_rows_kernel<bf16, 1>, grid, block, sm, a);
        return;
    }
    const CUtensorMap &mc = buf_map(pm, a.cache, l.ldc, l.ldc, a.seq, LG_WD_S);
    if (form == 0) {
        const int hpg = p.heads / p.kv_heads;
        const dim3 grid(l.C, p.kv_heads, (n * hpg + 15) / 16), block(LG_WD_THREADS);
        const size_t sm = lg_win_dec_smem(p.maps, l.dimp, l.vdp);
        if (!two) launch_k(e, lg_win_dec_attn_kernel<1, 4>, grid, block, sm, mc, a);
        else if (l.vdp <= 128) launch_k(e, lg_win_dec_attn_kernel<2, 4>, grid, block, sm, mc, a);
        else launch_k(e, lg_win_dec_attn_kernel<2, 8>, grid, block, sm, mc, a);
        if (two) launch_k(e, lg_win_merge_kernel<2>, dim3(n * p.heads), dim3(LG_WM_THREADS), 0, a, l.C);
        else launch_k(e, lg_win_merge_kernel<1>, dim3(n * p.heads), dim3(LG_WM_THREADS), 0, a, l.C);
        return;
    }
    const CUtensorMap &mq = buf_map(pm, a.q, l.q_cols, l.q_cols, q_rows, LG_WP_Q);
    const dim3 grid((n + LG_WP_Q - 1) / LG_WP_Q, p.heads);
    if (two) launch_k(e, lg_win_pf_attn_kernel<2>, grid, dim3(lg_win_pf_threads<2>()), lg_win_pf_smem(2, l.dimp, l.vdp), mq, mc, a);
    else launch_k(e, lg_win_pf_attn_kernel<1>, grid, dim3(lg_win_pf_threads<1>()), lg_win_pf_smem(1, l.dimp, l.vdp), mq, mc, a);
}

// The mixer of layer l with the state of slot `slot`: projection rows b.pj -> the first columns of b.at.  Kernel classes: C_ATTN the
// attention / state-space kernels, C_PLE the convolution and the gated norm around them.
void seq_mixer(Engine *e, const struct kvcache *kv, const PlanLayer &l, int slot, const Pass &p, int only) {
    PlanBuf &b = *p.b;
    const struct lg_plan_layer &q = l.p;
    const SeqBlock sb = seq_block(l, e->f32);
    uint8_t *blk = (uint8_t *)kv->v[slot];
    const bool f32_rows = !p.wide || e->f32;
    LgConvArgs c{};
    c.src = b.pj; c.ld = l.in.rows; c.ch0 = l.ch0; c.nch = l.nch; c.w = l.conv_w; c.bias = l.conv_b; c.taps = q.taps;
    c.ring = blk + sb.ring; c.mask = l.mask; c.pos = p.pos; c.M = p.n;
    if (q.mixer == LG_MIX_GROUPED) {
        uint8_t *rows = (uint8_t *)kv->k[slot];
        c.o[0] = {l.q_cols, b.q, l.q_cols, 0};
        c.o[1] = {l.nch, rows, l.ldc, kv->seq[slot]};
        if (only & C_PLE) launch_conv(e, c, f32_rows);
        if (!(only & C_ATTN)) return;
        LgWinArgs a{};
        a.q = b.q; a.cache = rows; a.seq = kv->seq[slot]; a.pos = p.pos; a.out = b.at; a.ldo = l.o.ldk;
        launch_win(e, l, e->f32 ? 1 : p.wide ? (l.chunked ? 2 : 1) : l.rt ? 0 : 1, p.n, b.cap, a);
        return;
    }
    const int inner = q.heads * l.vdp;
    float *state = (float *)(blk + sb.state);
    LgSsmStepArgs s{};
    s.src = b.pj; s.ld = l.in.rows; s.ch0 = l.ch0; s.dt_off = l.dt_off; s.w = l.conv_w; s.bias = l.conv_b; s.taps = q.taps; s.nch = l.nch;
    s.ring = blk + sb.ring; s.dt_ring = (float *)(blk + sb.dt); s.mask = l.mask; s.dt_bias = l.dt_bias; s.a_log = l.a_log; s.d = l.d;
    s.state = state; s.heads = q.heads; s.vdp = l.vdp; s.np = l.np; s.groups = q.groups; s.ctl = seq_ctl(kv); s.pos = p.pos; s.M = p.n; s.y = b.y; s.ldy = inner;
    LgGatedNormArgs g{};
    g.y = b.y; g.ldy = inner; g.z = b.pj; g.ldz = l.in.rows; g.w = l.gnorm; g.vd = q.vdim; g.vdp = l.vdp; g.n = q.heads * q.vdim / q.norm_groups; g.eps = l.eps;
    g.out = b.at; g.ldo = l.o.ldk;
    if (p.wide) {
        if (p.first && p.pos0 > 0 && (only & C_ATTN)) {          // up to the block's start: states of the narrow block before it
            LgSsmStepArgs r = s;
            r.M = 0;
            launch_ssm_step(e, l, r, false);
        }
        c.o[0] = {l.nch, b.cv, l.nch, 0};
        c.silu = 1;
        if (only & C_PLE) launch_conv(e, c, f32_rows);
        const float *dt = e->f32 ? b.pj + l.dt_off : b.dt;
        const int ld_dt = e->f32 ? l.in.rows : l.in.rows - l.dt_off;
        if (!(only & C_ATTN)) { }
        else if (l.chunked && !e->f32) launch_ssd(e, l, p.n, b.cap, b.cv, dt, ld_dt, b, state, p.pos0 == 0, b.y, inner);
        else {
            s.src = b.cv; s.ld = l.nch; s.dt_src = dt; s.ld_dt = ld_dt; s.fresh = p.pos0 == 0;
            launch_ssm_step(e, l, s, true);
        }
    } else if (only & C_ATTN) launch_ssm_step(e, l, s, false);
    if (only & C_PLE) launch_gated_norm(e, p.n, q.norm_groups, g, f32_rows);
}

// x in place -> every layer run -> (with final_norm) the normed rows in b->h and, narrow, in e->hidden
void seq_layers(Engine *e, const struct kvcache *kv, const Pass &p, bool final_norm, int only) {
    PlanModel *pm = e->plan;
    PlanBuf &b = *p.b;
    const struct lg_plan *P = pm->plan;
    const int W = P->width, ldh = up(W, 64), n_runs = (int)pm->runs.size();
    if (only & C_MISC) launch_k(e, lg_seq_begin_kernel, dim3(1), dim3(32), 0, seq_ctl(kv), p.pos, p.n, p.wide ? 1 : 0, e->err);
    LgRowNormArgs r{};
    r.x = b.x; r.ldx = W; r.n = W; r.eps = P->norm_eps; r.center = P->norm_kind == LG_NORM_LAYER; r.ldy = ldh; r.y = b.h; r.ldyf = W; r.ld_add = up(W, 32);
    // x += the layer before (none at the first); the vector of a pass that begins; norms of the layer behind
    auto next = [&](int i) {
        const bool end = i == n_runs;
        const PlanLayer *l = end ? nullptr : &pm->L[pm->runs[i].layer];
        r.add = i ? b.o : nullptr;
        r.bias = end ? nullptr : pm->runs[i].step;
        r.norm_w = end ? (final_norm ? pm->out_norm : nullptr) : l->norm1;
        r.norm_w2 = end ? nullptr : l->norm2; r.y2 = r.norm_w2 ? b.h2 : nullptr;
        r.yf = end && final_norm && !p.wide ? e->hidden : nullptr;
        if (only & C_NORM) launch_row_norm_par(e, p.n, r);
    };
    next(0);
    for (int i = 0; i < n_runs; i++) {
        const PlanLayer &l = pm->L[pm->runs[i].layer];
        uint8_t *act = (uint8_t *)b.at + (size_t)l.act_off * (e->f32 ? 4 : 2);
        if (e->f32) {
            if (only & C_QKV) launch_f32(e, l.in, b.h, ldh, p.n, b.pj, l.in.rows);
            if (l.p.ff && (only & C_QKV)) {
                launch_f32(e, l.gu, b.h2, ldh, p.n, b.gu, l.gu.rows);
                launch_k(e, lg_dn_relu2_rows, dim3((l.gu.rows + 255) / 256, p.n), dim3(256), 0, (const float *)b.gu, l.gu.rows, l.gu.rows, (float *)act, l.o.ldk);
            }
        } else if (p.wide) {
            if (only & C_QKV) {
                LgDnGemmArgs a{};
                a.f32_from = l.dt_off; a.out2 = b.dt; a.ldo2 = l.in.rows - l.dt_off;
                launch_dn_gemm<DN_G_BF16>(e, l.in, b.h, ldh, b.cap, p.n, b.pj, l.in.rows, a);
            }
            if (l.p.ff && (only & C_GATEUP)) launch_dn_gemm<DN_G_RELU2>(e, l.gu, b.h2, ldh, b.cap, p.n, act, l.o.ldk);
        } else if (only & C_QKV) {
            LgDnGemvArgs a{};
            a.x = (const bf16 *)b.h; a.x2 = (const bf16 *)b.h2; a.ldx = ldh; a.M = p.n; a.split_tile = l.in_rows / 16; a.out = b.pj; a.ldo = l.in.rows;
            a.outh = (bf16 *)act; a.ldoh = l.o.ldk;
            launch_dn_gemv<DN_PAIR, false>(e, l.inup, a);
        }
        seq_mixer(e, kv, l, pm->runs[i].slot, p, only);
        if (only & C_O) project(e, l.o, b.at, l.o.ldk, p, b.o);
        next(i + 1);
    }
}
