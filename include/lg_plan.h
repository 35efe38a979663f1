/* lg_plan.h -- layer plans: the description of a model whose layers are listed one by one, each with its own mixer,
 * sizes and constants, instead of being one block repeated with two kinds of attention.
 *
 * A plan is read from the metadata of an opened model, under the model's architecture prefix like every other
 * hyper-parameter:
 *
 *   block_count, embedding_length, vocab_size            u32
 *   block.form                                           string   "sandwich" (default) or "parallel"
 *   norm.kind                                            string   "layer" (mean taken off) or "rms"
 *   norm.epsilon, residual_multiplier                    f32
 *   norm.weight_offset                                   f32      added to every stored weight of a model-wide norm (default 0)
 *   logit_scale                                          f32      (default 1)
 *   feed_forward.activation                              string   "relu" (gated: relu(gate) * up) or "relu2" (square of relu, no gate)
 *   loop.start, loop.stop, loop.times                    u32      layers start .. stop-1 run `times` times in a row (default: once)
 *   layer.mixer                                          i32[]    enum lg_mixer
 *   feed_forward_length                                  i32[]    0 = the layer has no feed-forward
 * Per-layer lists a mixer does not use may be absent:
 *   latent attention: attention.head_count, attention.key_length (unrotated part), attention.rope_length,
 *   attention.value_length, attention.q_rank, attention.kv_rank, attention.kv_from (own index = none),
 *   rope.dimension_count                                 i32[]
 *   attention.scale, rope.freq_base                      f32[]
 *   grouped attention: attention.head_count, attention.head_count_kv, attention.key_length (per map), attention.value_length,
 *   attention.maps (softmax maps per head: 1, or 2 = their difference), attention.window (0 = everything), conv.taps   i32[]
 *   attention.scale, attention.diff                      f32[]
 *   state-space (Mamba-2): ssm.head_count, ssm.value_length, ssm.state_size, ssm.group_count, ssm.norm_groups, conv.taps   i32[]
 *
 * A sandwich layer does  x += m * norm(mixer(norm(x) w1)) w1b,  then  x += m * norm(ff(norm(x) w2)) w2b.
 * A parallel layer does  x += mixer(norm(x) w1) + ff(norm(x) w2), both of the same x.
 */
#ifndef LG_PLAN_H
#define LG_PLAN_H

#include "lg_abi.h"

#ifdef __cplusplus
extern "C" {
#endif

#define LG_CONV_MAX_TAPS 16

enum lg_mixer { LG_MIX_LATENT = 1, LG_MIX_GROUPED = 2, LG_MIX_SSM = 3 };
enum lg_norm_kind { LG_NORM_RMS = 0, LG_NORM_LAYER = 1 };
enum lg_act { LG_ACT_RELU = 0, LG_ACT_RELU2 = 1 };
enum lg_form { LG_FORM_SANDWICH = 0, LG_FORM_PARALLEL = 1 };

struct lg_plan_layer {
    int   mixer;                       /* enum lg_mixer */
    int   heads, dim, rot_dim, vdim;   /* per head: unrotated and rotated query/key sizes, value size */
    int   q_rank, kv_rank;             /* widths of the query latent and of the cached latent */
    int   kv_src;                      /* layer whose cached rows this layer reads (its own index: it writes them) */
    int   rot_dims;                    /* leading dimensions of the rotated part that are rotated (interleaved pairs) */
    float scale, rot_base;
    int   ff;                          /* 0: no feed-forward */
    int   kv_heads, maps, window;      /* grouped attention: key/value heads, softmax maps, positions seen (0: all) */
    int   taps;                        /* of the short convolution after the projections */
    float diff;                        /* two maps: constant part of the second one's weight */
    int   state, groups, norm_groups;  /* state-space: state size, groups of B / C, groups of the gated norm */
};

struct lg_plan {
    int   n_layer, width, vocab;
    int   norm_kind, act;
    float norm_eps, residual_mult;
    struct lg_plan_layer *layer;
    int   form;                        /* enum lg_form */
    float norm_offset, logit_scale;
    int   loop_start, loop_stop, loop_times;
};

/* Layer runs: a looped layer counts once per pass.  Run r executes layer lg_plan_run_layer(p, r, &pass); pass = number of the loop
 * pass that begins with this run, -1 where none does.  Every run has cache and state of its own. */
int  lg_plan_runs(const struct lg_plan *p);
int  lg_plan_run_layer(const struct lg_plan *p, int run, int *pass);

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
