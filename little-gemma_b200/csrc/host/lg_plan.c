/* lg_plan.c -- layer plans from an opened model's metadata (keys: lg_plan.h). */
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
static const void *array_of(const struct gguf_context *g, const char *leaf, uint32_t type, int n) {
    const struct gguf_meta *kv = key(g, leaf);
    if (kv && kv->type == GGUF_TYPE_ARRAY && kv->value.arr.type == type && kv->value.arr.n == (uint64_t)n) return kv->value.arr.data;
    fprintf(stderr, "plan: %s is missing or does not list %d layers\n", leaf, n);
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
    const char *nk = scalar_s(g, "norm.kind", "rms"), *act = scalar_s(g, "feed_forward.activation", "relu");
    p->norm_kind = !strcmp(nk, "layer") ? LG_NORM_LAYER : LG_NORM_RMS;
    p->act = LG_ACT_RELU;
    if (p->n_layer <= 0 || p->n_layer > 4096 || p->width <= 0 || p->vocab <= 0 || strcmp(act, "relu") || (strcmp(nk, "layer") && strcmp(nk, "rms"))) {
        fprintf(stderr, "plan: %d layers, width %d, vocabulary %d, norm '%s', activation '%s' is not a usable model\n", p->n_layer, p->width, p->vocab, nk, act);
        lg_plan_free(p);
        return NULL;
    }
    const int n = p->n_layer;
    p->layer = calloc((size_t)n, sizeof *p->layer);
    static const char *const ik[] = {"layer.mixer", "attention.head_count", "attention.key_length", "attention.rope_length", "attention.value_length",
                                     "attention.q_rank", "attention.kv_rank", "attention.kv_from", "rope.dimension_count", "feed_forward_length"};
    const int32_t *iv[10];
    const float *scale = array_of(g, "attention.scale", GGUF_TYPE_FLOAT32, n), *base = array_of(g, "rope.freq_base", GGUF_TYPE_FLOAT32, n);
    int ok = p->layer && scale && base;
    for (int i = 0; i < 10 && ok; i++) ok = (iv[i] = array_of(g, ik[i], GGUF_TYPE_INT32, n)) != NULL;
    if (!ok) { lg_plan_free(p); return NULL; }
    for (int L = 0; L < n; L++) {
        struct lg_plan_layer *l = &p->layer[L];
        l->mixer = iv[0][L]; l->heads = iv[1][L]; l->dim = iv[2][L]; l->rot_dim = iv[3][L]; l->vdim = iv[4][L];
        l->q_rank = iv[5][L]; l->kv_rank = iv[6][L]; l->kv_src = iv[7][L]; l->rot_dims = iv[8][L]; l->ff = iv[9][L];
        l->scale = scale[L]; l->rot_base = base[L];
        if (l->mixer != LG_MIX_LATENT) return bad(p, L, "unknown mixer"), NULL;
        if (l->heads < 1 || l->dim < 1 || l->rot_dim < 0 || l->vdim < 1 || l->q_rank < 1 || l->kv_rank < 1 || l->ff < 0 || !(l->scale > 0))
            return bad(p, L, "a size is out of range"), NULL;
        if (l->rot_dims < 0 || l->rot_dims > l->rot_dim || l->rot_dims % 2) return bad(p, L, "the rotated dimensions are not an even part of the rotated key part"), NULL;
        if (l->kv_src < 0 || l->kv_src > L) return bad(p, L, "reads the cache of a layer that has not run"), NULL;
        const struct lg_plan_layer *s = &p->layer[l->kv_src];
        if (s->kv_src != l->kv_src || s->kv_rank != l->kv_rank || s->rot_dim != l->rot_dim || s->rot_dims != l->rot_dims || s->rot_base != l->rot_base)
            return bad(p, L, "the cache it reads has another shape or rotation"), NULL;
    }
    return p;
}
