/* lg_plan.h -- layer plans: the description of a model whose layers are listed one by one, each with its own mixer,
 * sizes and constants, instead of being one block repeated with two kinds of attention.
 *
 * A plan is read from the metadata of an opened model, under the model's architecture prefix like every other
 * hyper-parameter:
 *
 *   block_count, embedding_length, vocab_size            u32
 *   norm.kind                                            string   "layer" (mean taken off) or "rms"
 *   norm.epsilon, residual_multiplier                    f32
 *   feed_forward.activation                              string   "relu"
 *   layer.mixer                                          i32[]    enum lg_mixer
 *   feed_forward_length                                  i32[]    0 = the layer has no feed-forward
 *   latent attention: attention.head_count, attention.key_length (unrotated part), attention.rope_length,
 *   attention.value_length, attention.q_rank, attention.kv_rank, attention.kv_from (own index = none),
 *   rope.dimension_count                                 i32[]
 *   attention.scale, rope.freq_base                      f32[]
 *
 * A layer does  x += m * norm(mixer(norm(x) w1)) w1b,  then  x += m * norm(ff(norm(x) w2)) w2b.
 */
#ifndef LG_PLAN_H
#define LG_PLAN_H

#include "lg_abi.h"

#ifdef __cplusplus
extern "C" {
#endif

enum lg_mixer { LG_MIX_LATENT = 1 };
enum lg_norm_kind { LG_NORM_RMS = 0, LG_NORM_LAYER = 1 };
enum lg_act { LG_ACT_RELU = 0 };

struct lg_plan_layer {
    int   mixer;                       /* enum lg_mixer */
    int   heads, dim, rot_dim, vdim;   /* per head: unrotated and rotated query/key sizes, value size */
    int   q_rank, kv_rank;             /* widths of the query latent and of the cached latent */
    int   kv_src;                      /* layer whose cached rows this layer reads (its own index: it writes them) */
    int   rot_dims;                    /* leading dimensions of the rotated part that are rotated (interleaved pairs) */
    float scale, rot_base;
    int   ff;                          /* 0: no feed-forward */
};

struct lg_plan {
    int   n_layer, width, vocab;
    int   norm_kind, act;
    float norm_eps, residual_mult;
    struct lg_plan_layer *layer;
};

/* Whether the model is described by a plan. */
int  lg_plan_present(const struct gguf_context *g);
/* Read and validate; NULL after a message on stderr. */
struct lg_plan *lg_plan_read(const struct gguf_context *g);
void lg_plan_free(struct lg_plan *p);

/* Open a checkpoint folder (config.json + model.safetensors) as a model container: tensors under this library's names
 * (blk.<layer>.<leaf>.weight), hyper-parameters as metadata.  The architecture named in config.json picks the reader.
 * NULL after a message on stderr.  Freed with free_gguf. */
struct gguf_context *load_checkpoint(const char *dir);
/* A GGUF file or a checkpoint folder. */
struct gguf_context *load_model(const char *path);

#ifdef __cplusplus
}
#endif
#endif /* LG_PLAN_H */
