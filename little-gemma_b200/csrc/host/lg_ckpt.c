/* lg_ckpt.c -- checkpoint folders (config.json + model.safetensors) opened as model containers.
 *
 * A safetensors file is an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets) and the
 * data, which is mapped read-only.  The reader of the architecture named in config.json turns the configuration into the
 * metadata keys the model set-up reads (lg_plan.h lists them) and gives the tensors this library's names, so everything
 * behind the container -- set-up, cache, engine -- is the same whatever file the model came from.
 */
#define _GNU_SOURCE
#include <ctype.h>
#include <fcntl.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>
#include "lg_host.h"
#include "lg_plan.h"

/* ---- JSON ------------------------------------------------------------------------------- */

enum { J_NULL, J_BOOL, J_NUM, J_STR, J_ARR, J_OBJ };
struct json {
    int type;
    double num;                         /* J_NUM, J_BOOL */
    char *str;                          /* J_STR */
    char *key;                          /* name of this member, in an object */
    struct json *child, *next;          /* J_ARR, J_OBJ: members in order */
};
struct jcur { const char *p, *end; int bad, depth; };

static void json_free(struct json *j) {
    while (j) {
        struct json *n = j->next;
        json_free(j->child);
        free(j->str); free(j->key); free(j);
        j = n;
    }
}
static void jspace(struct jcur *c) { while (c->p < c->end && strchr(" \t\r\n", *c->p) && *c->p) c->p++; }
static int jtake(struct jcur *c, char ch) {
    jspace(c);
    if (c->p < c->end && *c->p == ch) { c->p++; return 1; }
    return 0;
}
static char *jstring(struct jcur *c) {
    if (!jtake(c, '"')) { c->bad = 1; return NULL; }
    char *out = malloc((size_t)(c->end - c->p) + 1), *o = out;
    /* (sized for the worst case, then trimmed) */
    while (out && c->p < c->end && *c->p != '"') {
        if (*c->p != '\\') { *o++ = *c->p++; continue; }
        if (++c->p >= c->end) break;
        char ch = *c->p++;
        switch (ch) {
        case 'n': *o++ = '\n'; break; case 't': *o++ = '\t'; break; case 'r': *o++ = '\r'; break;
        case 'b': *o++ = '\b'; break; case 'f': *o++ = '\f'; break;
        case 'u': {
            unsigned v = 0;
            for (int i = 0; i < 4; i++) {
                if (c->p >= c->end || !isxdigit((unsigned char)*c->p)) { c->bad = 1; break; }
                char h = *c->p++;
                v = v * 16 + (unsigned)(h <= '9' ? h - '0' : (h | 32) - 'a' + 10);
            }
            if (v < 0x80) *o++ = (char)v;
            else if (v < 0x800) { *o++ = (char)(0xC0 | v >> 6); *o++ = (char)(0x80 | (v & 63)); }
            else { *o++ = (char)(0xE0 | v >> 12); *o++ = (char)(0x80 | ((v >> 6) & 63)); *o++ = (char)(0x80 | (v & 63)); }
            break;
        }
        default: *o++ = ch;
        }
    }
    if (!out || c->p >= c->end) { c->bad = 1; free(out); return NULL; }
    c->p++;
    *o = 0;
    char *fit = realloc(out, (size_t)(o - out) + 1);
    return fit ? fit : out;
}
static struct json *jvalue(struct jcur *c) {
    struct json *j = calloc(1, sizeof *j);
    jspace(c);
    if (!j || c->p >= c->end || ++c->depth > 64) { c->bad = 1; return j; }
    if (*c->p == '{' || *c->p == '[') {
        const int obj = *c->p++ == '{';
        const char close = obj ? '}' : ']';
        struct json **tail = &j->child;
        j->type = obj ? J_OBJ : J_ARR;
        if (!jtake(c, close))
            do {
                char *key = obj ? jstring(c) : NULL;
                if (obj && (c->bad || !jtake(c, ':'))) { free(key); c->bad = 1; break; }
                struct json *v = jvalue(c);
                if (!v) { free(key); break; }
                v->key = key;
                *tail = v; tail = &v->next;
                if (c->bad) break;
                if (jtake(c, close)) { c->depth--; return j; }
                if (!jtake(c, ',')) c->bad = 1;
            } while (!c->bad);
    } else if (*c->p == '"') {
        j->type = J_STR;
        j->str = jstring(c);
    } else if (c->end - c->p >= 4 && !strncmp(c->p, "true", 4)) { j->type = J_BOOL; j->num = 1; c->p += 4; }
    else if (c->end - c->p >= 5 && !strncmp(c->p, "false", 5)) { j->type = J_BOOL; c->p += 5; }
    else if (c->end - c->p >= 4 && !strncmp(c->p, "null", 4)) { j->type = J_NULL; c->p += 4; }
    else {
        char buf[64];
        size_t n = 0;
        while (c->p + n < c->end && n < sizeof buf - 1 && (isdigit((unsigned char)c->p[n]) || (c->p[n] && strchr("+-.eE", c->p[n])))) { buf[n] = c->p[n]; n++; }
        buf[n] = 0;
        char *e = NULL;
        j->type = J_NUM;
        j->num = strtod(buf, &e);
        if (!n || *e) c->bad = 1;
        c->p += n;
    }
    c->depth--;
    return j;
}
static struct json *json_parse(const char *text, size_t n) {
    struct jcur c = {text, text + n, 0, 0};
    struct json *j = jvalue(&c);
    jspace(&c);
    if (c.bad || c.p != c.end) { json_free(j); return NULL; }
    return j;
}
static const struct json *jget(const struct json *o, const char *key) {
    if (!o || o->type != J_OBJ) return NULL;
    for (const struct json *v = o->child; v; v = v->next) if (v->key && !strcmp(v->key, key)) return v;
    return NULL;
}
/* a required number; *ok turns 0 with a message when it is missing */
static double jnum(const struct json *o, const char *key, const char *where, int *ok) {
    const struct json *v = jget(o, key);
    if (v && v->type == J_NUM) return v->num;
    if (*ok) fprintf(stderr, "checkpoint: %s has no number '%s'\n", where, key);
    *ok = 0;
    return 0;
}
static int jint(const struct json *o, const char *key, const char *where, int *ok) {
    const double d = jnum(o, key, where, ok);
    const int i = d >= -2147483647.0 && d <= 2147483647.0 ? (int)d : 0;
    if (*ok && (double)i != d) { fprintf(stderr, "checkpoint: %s: '%s' = %g is not an integer\n", where, key, d); *ok = 0; }
    return i;
}

/* ---- metadata --------------------------------------------------------------------------- */

static struct gguf_meta *meta_new(struct gguf_context *g, const char *prefix, const char *leaf, uint32_t type) {
    struct gguf_meta *m = realloc(g->meta, (g->header.num_meta + 1) * sizeof *m);
    if (!m) { fprintf(stderr, "checkpoint: out of memory\n"); exit(1); }
    g->meta = m;
    m += g->header.num_meta++;
    memset(m, 0, sizeof *m);
    if (asprintf(&m->key, "%s.%s", prefix, leaf) < 0) exit(1);
    m->type = type;
    return m;
}
static void meta_u32(struct gguf_context *g, const char *p, const char *leaf, uint32_t v) { meta_new(g, p, leaf, GGUF_TYPE_UINT32)->value.u32 = v; }
static void meta_f32(struct gguf_context *g, const char *p, const char *leaf, double v) { meta_new(g, p, leaf, GGUF_TYPE_FLOAT32)->value.f32 = (float)v; }
static void meta_str(struct gguf_context *g, const char *p, const char *leaf, const char *v) { meta_new(g, p, leaf, GGUF_TYPE_STRING)->value.str = strdup(v); }
/* a per-layer array of 4-byte elements; returns its storage */
static void *meta_arr(struct gguf_context *g, const char *p, const char *leaf, uint32_t type, int n) {
    void *data = calloc((size_t)(n > 0 ? n : 1), 4);
    if (!data) { fprintf(stderr, "checkpoint: out of memory\n"); exit(1); }
    struct gguf_meta *m = meta_new(g, p, leaf, GGUF_TYPE_ARRAY);
    m->value.arr.type = type; m->value.arr.n = (uint64_t)n; m->value.arr.data = data;
    return data;
}

/* ---- architectures ---------------------------------------------------------------------- */

struct rename { const char *from, *to; };
struct ckpt_arch {
    const char *name;                   /* config.json 'architecture' */
    const char *prefix;                 /* metadata prefix and general.architecture */
    int (*configure)(struct gguf_context *g, const char *prefix, const struct json *cfg);      /* 0 / -1 */
    const char *layer_prefix;           /* tensors of layer i start with <layer_prefix><i>. */
    const struct rename *layer, *model; /* leaf names inside a layer, and names outside of the layers */
};

/* Mubopel: latent attention in every layer (queries and keys/values through latents, one rotated key part shared by the
 * heads, a sink per head, an output gate), layers that borrow the latent rows of an earlier one, dense ReLU-gated
 * feed-forward, layer norm before and after each sublayer, scaled residual additions, tied output head. */
static int mubopel_configure(struct gguf_context *g, const char *prefix, const struct json *cfg) {
    int ok = 1;
    const struct json *layers = jget(cfg, "layers");
    int n = 0;
    if (layers && layers->type == J_ARR) for (const struct json *l = layers->child; l; l = l->next) n++;
    if (!n) { fprintf(stderr, "checkpoint: config.json lists no layers\n"); return -1; }
    meta_u32(g, prefix, "block_count", (uint32_t)n);
    meta_u32(g, prefix, "embedding_length", (uint32_t)jint(cfg, "width", "config.json", &ok));
    meta_u32(g, prefix, "vocab_size", (uint32_t)jint(cfg, "vocab", "config.json", &ok));
    meta_f32(g, prefix, "residual_multiplier", jnum(cfg, "residual_mult", "config.json", &ok));
    meta_f32(g, prefix, "norm.epsilon", jnum(jget(cfg, "norm"), "eps", "norm", &ok));
    meta_str(g, prefix, "norm.kind", "layer");
    meta_str(g, prefix, "feed_forward.activation", "relu");
    static const struct { const char *leaf, *key; } ints[] = {
        {"attention.head_count", "heads"}, {"attention.key_length", "dim"}, {"attention.rope_length", "rot_dim"},
        {"attention.value_length", "vdim"}, {"attention.q_rank", "q_rank"}, {"attention.kv_rank", "kv_rank"}};
    enum { NI = sizeof ints / sizeof *ints };
    int32_t *iv[NI];
    for (int i = 0; i < NI; i++) iv[i] = meta_arr(g, prefix, ints[i].leaf, GGUF_TYPE_INT32, n);
    int32_t *mixer = meta_arr(g, prefix, "layer.mixer", GGUF_TYPE_INT32, n), *from = meta_arr(g, prefix, "attention.kv_from", GGUF_TYPE_INT32, n);
    int32_t *dims = meta_arr(g, prefix, "rope.dimension_count", GGUF_TYPE_INT32, n), *ff = meta_arr(g, prefix, "feed_forward_length", GGUF_TYPE_INT32, n);
    float *scale = meta_arr(g, prefix, "attention.scale", GGUF_TYPE_FLOAT32, n), *base = meta_arr(g, prefix, "rope.freq_base", GGUF_TYPE_FLOAT32, n);
    int L = 0;
    for (const struct json *l = layers->child; l; l = l->next, L++) {
        char where[32];
        snprintf(where, sizeof where, "layer %d", L);
        const struct json *type = jget(l, "type"), *mx = jget(l, "mixer"), *mlp = jget(l, "mlp"), *rot = jget(mx, "rot");
        if (!type || type->type != J_STR || strcmp(type->str, "latent_attention")) {
            fprintf(stderr, "checkpoint: %s has a mixer this library does not know: '%s'\n", where, type && type->type == J_STR ? type->str : "?");
            return -1;
        }
        mixer[L] = LG_MIX_LATENT;
        for (int i = 0; i < NI; i++) iv[i][L] = jint(mx, ints[i].key, where, &ok);
        from[L] = jget(mx, "kv_from") && jget(mx, "kv_from")->type != J_NULL ? jint(mx, "kv_from", where, &ok) : L;
        scale[L] = (float)jnum(mx, "scale", where, &ok);
        dims[L] = rot ? jint(rot, "dims", where, &ok) : 0;
        base[L] = rot ? (float)jnum(rot, "base", where, &ok) : 1.0f;
        if (mlp && mlp->type == J_OBJ) {
            const struct json *kind = jget(mlp, "kind");
            if (!kind || kind->type != J_STR || strcmp(kind->str, "dense")) { fprintf(stderr, "checkpoint: %s has an unknown kind of feed-forward\n", where); return -1; }
            ff[L] = jint(mlp, "ff", where, &ok);
        }
    }
    return ok ? 0 : -1;
}
static const struct rename mubopel_layer[] = {
    {"norm1", "attn_norm"}, {"norm1b", "post_attention_norm"}, {"norm2", "ffn_norm"}, {"norm2b", "post_ffw_norm"},
    {"mix.dq", "attn_q_a"}, {"mix.dq.norm", "attn_q_a_norm"}, {"mix.uq", "attn_q_b"},
    {"mix.dkv", "attn_kv_a"}, {"mix.dkv.norm", "attn_kv_a_norm"}, {"mix.uk", "attn_k_b"}, {"mix.uv", "attn_v_b"},
    {"mix.sink", "attn_sinks"}, {"mix.g", "attn_gate"}, {"mix.o", "attn_output"},
    {"mlp.gate", "ffn_gate"}, {"mlp.up", "ffn_up"}, {"mlp.down", "ffn_down"}, {NULL, NULL}};
static const struct rename mubopel_model[] = {{"embed", "token_embd"}, {"final.norm", "output_norm"}, {NULL, NULL}};

/* Baporax: layers that add a mixer and a feed-forward (square of ReLU) of the same x, RMS norms stored as distances from 1; mixers are
 * Mamba-2 state-space layers and sliding-window differential attention with short convolutions on q, k and v; a stretch of layers
 * runs several times with a vector added before each pass; tied output head with scaled logits. */
enum { BAPORAX_MAPS = 2 };
static int jstr_is(const struct json *v, const char *s) { return v && v->type == J_STR && !strcmp(v->str, s); }
static int jset(const struct json *o, const char *key) { const struct json *v = jget(o, key); return v && v->type != J_NULL; }
static int baporax_configure(struct gguf_context *g, const char *prefix, const struct json *cfg) {
    int ok = 1, n = 0;
    const struct json *layers = jget(cfg, "layers"), *loop = jget(cfg, "loop");
    if (layers && layers->type == J_ARR) for (const struct json *l = layers->child; l; l = l->next) n++;
    if (!n) { fprintf(stderr, "checkpoint: config.json lists no layers\n"); return -1; }
    meta_u32(g, prefix, "block_count", (uint32_t)n);
    meta_u32(g, prefix, "embedding_length", (uint32_t)jint(cfg, "width", "config.json", &ok));
    meta_u32(g, prefix, "vocab_size", (uint32_t)jint(cfg, "vocab", "config.json", &ok));
    meta_f32(g, prefix, "logit_scale", jnum(cfg, "logit_scale", "config.json", &ok));
    meta_f32(g, prefix, "norm.epsilon", jnum(jget(cfg, "norm"), "eps", "norm", &ok));
    meta_f32(g, prefix, "norm.weight_offset", 1.0);
    meta_str(g, prefix, "norm.kind", "rms");
    meta_str(g, prefix, "block.form", "parallel");
    meta_str(g, prefix, "feed_forward.activation", "relu2");
    if (loop && loop->type == J_OBJ) {
        meta_u32(g, prefix, "loop.start", (uint32_t)jint(loop, "start", "loop", &ok));
        meta_u32(g, prefix, "loop.stop", (uint32_t)jint(loop, "stop", "loop", &ok));
        meta_u32(g, prefix, "loop.times", (uint32_t)jint(loop, "times", "loop", &ok));
    }
    enum { HEADS, DIM, VDIM, KV, MAPS, WINDOW, TAPS, S_HEADS, S_VDIM, S_STATE, S_GROUPS, S_NORM, MIXER, FF, NI };
    static const char *const leaf[NI] = {"attention.head_count", "attention.key_length", "attention.value_length", "attention.head_count_kv",
        "attention.maps", "attention.window", "conv.taps", "ssm.head_count", "ssm.value_length", "ssm.state_size", "ssm.group_count",
        "ssm.norm_groups", "layer.mixer", "feed_forward_length"};
    int32_t *iv[NI];
    for (int i = 0; i < NI; i++) iv[i] = meta_arr(g, prefix, leaf[i], GGUF_TYPE_INT32, n);
    float *scale = meta_arr(g, prefix, "attention.scale", GGUF_TYPE_FLOAT32, n), *diff = meta_arr(g, prefix, "attention.diff", GGUF_TYPE_FLOAT32, n);
    int L = 0;
    for (const struct json *l = layers->child; l; l = l->next, L++) {
        char where[32];
        snprintf(where, sizeof where, "layer %d", L);
        const struct json *type = jget(l, "type"), *mx = jget(l, "mixer"), *mlp = jget(l, "mlp");
        static const struct { const char *key; int to; } attn[] = {{"heads", HEADS}, {"dim", DIM}, {"vdim", VDIM}, {"kv_heads", KV}, {"conv", TAPS}, {NULL, 0}},
            ssm[] = {{"heads", S_HEADS}, {"vdim", S_VDIM}, {"state", S_STATE}, {"groups", S_GROUPS}, {"norm_groups", S_NORM}, {"conv", TAPS}, {NULL, 0}}, *f;
        if (jstr_is(type, "attention")) {
            iv[MIXER][L] = LG_MIX_GROUPED;
            iv[MAPS][L] = BAPORAX_MAPS;
            if (jset(mx, "mask")) {
                iv[WINDOW][L] = jint(jget(mx, "mask"), "size", where, &ok);
                if (iv[WINDOW][L] < 1) { fprintf(stderr, "checkpoint: %s sees no position\n", where); return -1; }
            }
            scale[L] = (float)jnum(mx, "scale", where, &ok);
            diff[L] = (float)jnum(mx, "diff", where, &ok);
            f = attn;
        } else if (jstr_is(type, "mamba2")) {
            iv[MIXER][L] = LG_MIX_SSM;
            f = ssm;
        } else {
            fprintf(stderr, "checkpoint: %s has a mixer this library does not know: '%s'\n", where, type && type->type == J_STR ? type->str : "?");
            return -1;
        }
        for (; f->key; f++) iv[f->to][L] = jint(mx, f->key, where, &ok);
        if (mlp && mlp->type == J_OBJ) {
            if (!jstr_is(jget(mlp, "kind"), "dense")) { fprintf(stderr, "checkpoint: %s has an unknown kind of feed-forward\n", where); return -1; }
            iv[FF][L] = jint(mlp, "ff", where, &ok);
        }
    }
    return ok ? 0 : -1;
}
static const struct rename baporax_layer[] = {
    {"norm1", "attn_norm"}, {"norm2", "ffn_norm"}, {"mlp.up", "ffn_up"}, {"mlp.down", "ffn_down"}, {"mix.o", "attn_output"},
    {"mix.q", "attn_q"}, {"mix.k", "attn_k"}, {"mix.v", "attn_v"}, {"mix.q.conv", "attn_q_conv"}, {"mix.k.conv", "attn_k_conv"},
    {"mix.v.conv", "attn_v_conv"}, {"mix.lq1", "attn_lambda_q1"}, {"mix.lk1", "attn_lambda_k1"}, {"mix.lq2", "attn_lambda_q2"},
    {"mix.lk2", "attn_lambda_k2"}, {"mix.in", "ssm_in"}, {"mix.conv", "ssm_conv1d"}, {"mix.conv.b", "ssm_conv1d_bias"},
    {"mix.dt_bias", "ssm_dt_bias"}, {"mix.A_log", "ssm_a_log"}, {"mix.D", "ssm_d"}, {"mix.norm", "ssm_norm"}, {NULL, NULL}};
static const struct rename baporax_model[] = {{"embed", "token_embd"}, {"final.norm", "output_norm"}, {"loop.step", "loop_step"}, {NULL, NULL}};

static const struct ckpt_arch archs[] = {
    {"Mubopel", "mubopel", mubopel_configure, "l", mubopel_layer, mubopel_model},
    {"Baporax", "baporax", baporax_configure, "l", baporax_layer, baporax_model},
};

/* the library's name of a checkpoint tensor (caller frees), or NULL for one the architecture does not have */
static char *canonical(const struct ckpt_arch *a, const char *name) {
    const size_t np = strlen(a->layer_prefix);
    char *out = NULL, *end = NULL;
    for (const struct rename *r = a->model; r->from; r++)
        if (!strcmp(name, r->from)) return asprintf(&out, "%s.weight", r->to) < 0 ? NULL : out;
    if (strncmp(name, a->layer_prefix, np) || !isdigit((unsigned char)name[np])) return NULL;
    const long L = strtol(name + np, &end, 10);
    if (*end != '.') return NULL;
    for (const struct rename *r = a->layer; r->from; r++)
        if (!strcmp(end + 1, r->from)) return asprintf(&out, "blk.%ld.%s.weight", L, r->to) < 0 ? NULL : out;
    return NULL;
}

/* ---- opening ---------------------------------------------------------------------------- */

static struct json *read_json_file(const char *path) {
    FILE *f = fopen(path, "rb");
    if (!f) { fprintf(stderr, "checkpoint: cannot open %s\n", path); return NULL; }
    struct stat st;
    struct json *j = NULL;
    if (fstat(fileno(f), &st) == 0 && st.st_size > 0 && st.st_size < (1 << 28)) {
        char *text = malloc((size_t)st.st_size);
        if (text && fread(text, 1, (size_t)st.st_size, f) == (size_t)st.st_size) j = json_parse(text, (size_t)st.st_size);
        free(text);
    }
    fclose(f);
    if (!j) fprintf(stderr, "checkpoint: %s is not valid JSON\n", path);
    return j;
}

static int add_tensors(struct gguf_context *g, const struct ckpt_arch *a, const struct json *head) {
    size_t n = 0;
    for (const struct json *t = head->child; t; t = t->next) n++;
    g->tensors = calloc(n ? n : 1, sizeof *g->tensors);
    if (!g->tensors) return -1;
    for (const struct json *t = head->child; t; t = t->next) {
        if (!strcmp(t->key, "__metadata__")) continue;
        const struct json *dt = jget(t, "dtype"), *sh = jget(t, "shape"), *off = jget(t, "data_offsets");
        if (!dt || dt->type != J_STR || !sh || sh->type != J_ARR || !off || off->type != J_ARR || !off->child || !off->child->next) {
            fprintf(stderr, "checkpoint: malformed entry of tensor %s\n", t->key);
            return -1;
        }
        char *name = canonical(a, t->key);
        if (!name) { fprintf(stderr, "checkpoint: tensor %s is not part of a %s model\n", t->key, a->name); return -1; }
        struct gguf_tensor *q = &g->tensors[g->header.num_tensors++];
        q->name = name;
        size_t es;
        if (!strcmp(dt->str, "BF16")) { q->type = GGML_TYPE_BF16; es = 2; }
        else if (!strcmp(dt->str, "F16")) { q->type = GGML_TYPE_F16; es = 2; }
        else if (!strcmp(dt->str, "F32")) { q->type = GGML_TYPE_F32; es = 4; }
        else { fprintf(stderr, "checkpoint: tensor %s has unsupported type %s\n", t->key, dt->str); return -1; }
        uint64_t shape[4], elems = 1;
        for (const struct json *d = sh->child; d; d = d->next) {
            if (q->n_dims == 4 || d->type != J_NUM || d->num < 1 || d->num > 1e9) { fprintf(stderr, "checkpoint: tensor %s has an unusable shape\n", t->key); return -1; }
            shape[q->n_dims++] = (uint64_t)d->num;
            elems *= (uint64_t)d->num;
            if (elems > (uint64_t)g->data_size) { fprintf(stderr, "checkpoint: tensor %s is larger than the file\n", t->key); return -1; }
        }
        for (uint32_t d = 0; d < 4; d++) q->dims[d] = d < q->n_dims ? shape[q->n_dims - 1 - d] : 1;      /* innermost first */
        if (!q->n_dims) q->n_dims = 1;
        const double lo = off->child->num, hi = off->child->next->num;
        if (lo < 0 || hi < lo || hi > (double)g->data_size || (uint64_t)(hi - lo) != elems * es) {
            fprintf(stderr, "checkpoint: tensor %s lies outside the file or has the wrong size\n", t->key);
            return -1;
        }
        q->offset = (uint64_t)lo;
        q->data = (unsigned char *)g->data + q->offset;
    }
    return 0;
}

struct gguf_context *load_checkpoint(const char *dir) {
    char path[4096];
    snprintf(path, sizeof path, "%s/config.json", dir);
    struct json *cfg = read_json_file(path), *head = NULL;
    if (!cfg) return NULL;
    const struct json *an = jget(cfg, "architecture");
    const struct ckpt_arch *a = NULL;
    for (size_t i = 0; i < sizeof archs / sizeof *archs; i++)
        if (an && an->type == J_STR && !strcmp(an->str, archs[i].name)) a = &archs[i];
    if (!a) {
        fprintf(stderr, "checkpoint: %s: unknown architecture '%s'\n", path, an && an->type == J_STR ? an->str : "");
        json_free(cfg);
        return NULL;
    }
    struct gguf_context *g = calloc(1, sizeof *g);
    if (!g) { json_free(cfg); return NULL; }
    g->map_fd = -1;
    meta_str(g, "general", "architecture", a->prefix);
    int ok = a->configure(g, a->prefix, cfg) == 0;
    json_free(cfg);
    snprintf(path, sizeof path, "%s/model.safetensors", dir);
    struct stat st;
    if (ok) {
        g->map_fd = open(path, O_RDONLY);
        ok = g->map_fd >= 0 && fstat(g->map_fd, &st) == 0 && st.st_size > 8;
        if (!ok) fprintf(stderr, "checkpoint: cannot open %s\n", path);
    }
    if (ok) {
        void *base = mmap(NULL, (size_t)st.st_size, PROT_READ, MAP_PRIVATE, g->map_fd, 0);
        ok = base != MAP_FAILED;
        if (ok) { g->map_base = base; g->map_len = (size_t)st.st_size; }
    }
    if (ok) {
        const unsigned char *b = g->map_base;
        uint64_t n = 0;
        for (int i = 7; i >= 0; i--) n = n << 8 | b[i];
        ok = n <= g->map_len - 8 && (head = json_parse((const char *)b + 8, (size_t)n)) != NULL && head->type == J_OBJ;
        if (!ok) fprintf(stderr, "checkpoint: %s has no readable header\n", path);
        else {
            g->alignment = 1;
            g->data_offset = 8 + (size_t)n;
            g->data = (unsigned char *)g->map_base + g->data_offset;
            g->data_size = g->map_len - g->data_offset;
            ok = add_tensors(g, a, head) == 0;
        }
        json_free(head);
    }
    if (!ok) { free_gguf(g); return NULL; }
    return g;
}

struct gguf_context *load_model(const char *path) {
    struct stat st;
    if (stat(path, &st) == 0 && S_ISDIR(st.st_mode)) return load_checkpoint(path);
    return load_gguf(path);
}
