/* lg_plan.c -- layer plans from an opened model's metadata (keys: lg_plan.h). */
#include <stddef.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>
#include "lg_host.h"
#include "lg_plan.h"

static const struct gguf_meta *key(const struct gguf_context *g, const char *leaf) {
    char name[160];
    snprintf(name, sizeof name, "%s.%s", gguf_get_str(g, "general.architecture", ""), leaf);
    return gguf_find_meta(g, name);
}
static int scalar_i(const struct gguf_context *g, const char *leaf, int fb) {
    const struct gguf_meta *kv = key(g, leaf);
    return kv && (kv->type == GGUF_TYPE_UINT32 || kv->type == GGUF_TYPE_INT32) ? kv->value.i32 : fb;
}
static float scalar_f(const struct gguf_context *g, const char *leaf, float fb) {
    const struct gguf_meta *kv = key(g, leaf);
    return kv && kv->type == GGUF_TYPE_FLOAT32 ? kv->value.f32 : fb;
}
static const char *scalar_s(const struct gguf_context *g, const char *leaf, const char *fb) {
    const struct gguf_meta *kv = key(g, leaf);
    return kv && kv->type == GGUF_TYPE_STRING && kv->value.str ? kv->value.str : fb;
}
/* a per-layer list, or NULL when there is none; *ok turns 0 with a message when it is required or has another length */
static const void *array_of(const struct gguf_context *g, const char *leaf, uint32_t type, int n, int required, int *ok) {
    const struct gguf_meta *kv = key(g, leaf);
    if (!kv && !required) return NULL;
    if (kv && kv->type == GGUF_TYPE_ARRAY && kv->value.arr.type == type && kv->value.arr.n == (uint64_t)n) return kv->value.arr.data;
    fprintf(stderr, "plan: %s is missing or does not list %d layers\n", leaf, n);
    *ok = 0;
    return NULL;
}

int lg_plan_present(const struct gguf_context *g) { return g && key(g, "layer.mixer") != NULL; }

void lg_plan_free(struct lg_plan *p) { if (p) { free(p->layer); free(p); } }

static int bad(struct lg_plan *p, int L, const char *what) {
    fprintf(stderr, "plan: layer %d: %s\n", L, what);
    lg_plan_free(p);
    return 0;
}

struct lg_plan *lg_plan_read(const struct gguf_context *g) {
    struct lg_plan *p = calloc(1, sizeof *p);
    if (!p) return NULL;
    p->n_layer = scalar_i(g, "block_count", 0);
    p->width = scalar_i(g, "embedding_length", 0);
    p->vocab = scalar_i(g, "vocab_size", 0);
    p->norm_eps = scalar_f(g, "norm.epsilon", 1e-5f);
    p->residual_mult = scalar_f(g, "residual_multiplier", 1.0f);
    p->norm_offset = scalar_f(g, "norm.weight_offset", 0.0f);
    p->logit_scale = scalar_f(g, "logit_scale", 1.0f);
    const char *nk = scalar_s(g, "norm.kind", "rms"), *act = scalar_s(g, "feed_forward.activation", "relu"), *form = scalar_s(g, "block.form", "sandwich");
    p->norm_kind = !strcmp(nk, "layer") ? LG_NORM_LAYER : LG_NORM_RMS;
    p->act = !strcmp(act, "relu2") ? LG_ACT_RELU2 : LG_ACT_RELU;
    p->form = !strcmp(form, "parallel") ? LG_FORM_PARALLEL : LG_FORM_SANDWICH;
    if (p->n_layer <= 0 || p->n_layer > 4096 || p->width <= 0 || p->vocab <= 0 || (strcmp(act, "relu") && strcmp(act, "relu2")) ||
        (strcmp(nk, "layer") && strcmp(nk, "rms")) || (strcmp(form, "sandwich") && strcmp(form, "parallel"))) {
        fprintf(stderr, "plan: %d layers, width %d, vocabulary %d, norm '%s', activation '%s', form '%s' is not a usable model\n",
                p->n_layer, p->width, p->vocab, nk, act, form);
        lg_plan_free(p);
        return NULL;
    }
    const int n = p->n_layer;
    p->loop_start = scalar_i(g, "loop.start", 0);
    p->loop_stop = scalar_i(g, "loop.stop", 0);
    p->loop_times = scalar_i(g, "loop.times", 0);              /* 0: no loop */
    if (p->loop_times < 0 || (p->loop_times && (p->loop_start < 0 || p->loop_stop <= p->loop_start || p->loop_stop > n)) ||
        (p->loop_times && p->form != LG_FORM_PARALLEL) || (long long)p->loop_times * (p->loop_stop - p->loop_start) > 4096) {
        fprintf(stderr, "plan: layers %d .. %d, %d times, is not a usable loop\n", p->loop_start, p->loop_stop, p->loop_times);
        lg_plan_free(p);
        return NULL;
    }
    p->layer = calloc((size_t)n, sizeof *p->layer);
    /* every list with the member it fills; the first two are required */
    static const struct { const char *leaf; size_t at; } ik[] = {
#define AT(m) offsetof(struct lg_plan_layer, m)
        {"layer.mixer", AT(mixer)}, {"feed_forward_length", AT(ff)}, {"attention.head_count", AT(heads)}, {"attention.key_length", AT(dim)},
        {"attention.rope_length", AT(rot_dim)}, {"attention.value_length", AT(vdim)}, {"attention.q_rank", AT(q_rank)},
        {"attention.kv_rank", AT(kv_rank)}, {"attention.kv_from", AT(kv_src)}, {"rope.dimension_count", AT(rot_dims)},
        {"attention.head_count_kv", AT(kv_heads)}, {"attention.maps", AT(maps)}, {"attention.window", AT(window)}, {"conv.taps", AT(taps)},
        {"ssm.state_size", AT(state)}, {"ssm.group_count", AT(groups)}, {"ssm.norm_groups", AT(norm_groups)}},
      fk[] = {{"attention.scale", AT(scale)}, {"rope.freq_base", AT(rot_base)}, {"attention.diff", AT(diff)}},
      sk[] = {{"ssm.head_count", AT(heads)}, {"ssm.value_length", AT(vdim)}};
#undef AT
    int ok = p->layer != NULL;
    for (size_t i = 0; ok && i < sizeof ik / sizeof *ik; i++) {
        const int32_t *v = array_of(g, ik[i].leaf, GGUF_TYPE_INT32, n, i < 2, &ok);
        for (int L = 0; v && L < n; L++) memcpy((char *)&p->layer[L] + ik[i].at, &v[L], 4);
    }
    for (size_t i = 0; ok && i < sizeof fk / sizeof *fk; i++) {
        const float *v = array_of(g, fk[i].leaf, GGUF_TYPE_FLOAT32, n, 0, &ok);
        for (int L = 0; v && L < n; L++) memcpy((char *)&p->layer[L] + fk[i].at, &v[L], 4);
    }
    for (size_t i = 0; ok && i < sizeof sk / sizeof *sk; i++) {
        const int32_t *v = array_of(g, sk[i].leaf, GGUF_TYPE_INT32, n, 0, &ok);
        for (int L = 0; v && L < n; L++) if (p->layer[L].mixer == LG_MIX_SSM) memcpy((char *)&p->layer[L] + sk[i].at, &v[L], 4);
    }
    if (!ok) { lg_plan_free(p); return NULL; }
    for (int L = 0; L < n; L++) {
        struct lg_plan_layer *l = &p->layer[L];
        if (l->mixer < LG_MIX_LATENT || l->mixer > LG_MIX_SSM) return bad(p, L, "unknown mixer"), NULL;
        if (l->heads < 1 || l->vdim < 1 || l->ff < 0) return bad(p, L, "a size is out of range"), NULL;
        if ((l->mixer == LG_MIX_LATENT) != (p->form == LG_FORM_SANDWICH)) return bad(p, L, "a mixer this form of layer does not have"), NULL;
        if (l->mixer == LG_MIX_LATENT) {
            if (!key(g, "attention.kv_from")) return bad(p, L, "no list of cache owners"), NULL;
            if (l->dim < 1 || l->rot_dim < 0 || l->q_rank < 1 || l->kv_rank < 1 || !(l->scale > 0)) return bad(p, L, "a size is out of range"), NULL;
            if (l->rot_dims < 0 || l->rot_dims > l->rot_dim || l->rot_dims % 2) return bad(p, L, "the rotated dimensions are not an even part of the rotated key part"), NULL;
            if (l->kv_src < 0 || l->kv_src > L) return bad(p, L, "reads the cache of a layer that has not run"), NULL;
            const struct lg_plan_layer *s = &p->layer[l->kv_src];
            if (s->kv_src != l->kv_src || s->kv_rank != l->kv_rank || s->rot_dim != l->rot_dim || s->rot_dims != l->rot_dims || s->rot_base != l->rot_base)
                return bad(p, L, "the cache it reads has another shape or rotation"), NULL;
            continue;
        }
        l->kv_src = L;
        if (l->taps < 1 || l->taps > LG_CONV_MAX_TAPS) return bad(p, L, "the short convolution's length is out of range"), NULL;
        if (l->mixer == LG_MIX_GROUPED) {
            if (l->dim < 1 || l->kv_heads < 1 || l->heads % l->kv_heads || l->maps < 1 || l->maps > 2 || l->window < 0 || !(l->scale > 0))
                return bad(p, L, "a size is out of range"), NULL;
        } else if (l->state < 1 || l->groups < 1 || l->heads % l->groups || l->norm_groups < 1 || (l->heads * l->vdim) % l->norm_groups)
            return bad(p, L, "a size is out of range"), NULL;
    }
    return p;
}

int lg_plan_runs(const struct lg_plan *p) {
    return p->n_layer + (p->loop_times ? (p->loop_times - 1) * (p->loop_stop - p->loop_start) : 0);
}
int lg_plan_run_layer(const struct lg_plan *p, int run, int *pass) {
    if (pass) *pass = -1;
    if (!p->loop_times || run < p->loop_start) return run;
    const int len = p->loop_stop - p->loop_start, in = run - p->loop_start;
    if (in >= len * p->loop_times) return run - len * (p->loop_times - 1);
    if (pass && in % len == 0) *pass = in / len;
    return p->loop_start + in % len;
}
