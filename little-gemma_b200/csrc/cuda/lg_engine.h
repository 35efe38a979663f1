// lg_engine.h -- the engine's state and launch helpers, shared by the translation units of the backend: lg_engine.cu (the
// exported model API, sessions, graphs, the block-quantised models) and the layer-plan models (lg_plan.cu).
#ifndef LG_ENGINE_H
#define LG_ENGINE_H

#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <cmath>
#include <vector>
#include <map>
#include <string>
#include "lg_device.cuh"
#include "lg_host.h"
#include "lg_b200.h"

#define LG_CHECK(x) do { cudaError_t e_ = (x); if (e_ != cudaSuccess) { \
    fprintf(stderr, "lg_b200: CUDA error %s at %s:%d\n", cudaGetErrorString(e_), __FILE__, __LINE__); exit(1); } } while (0)

namespace lg {

struct Engine;
struct PlanModel;

// What one forward enqueues (flags of enqueue_forward and of a family's forward).
enum { F_HEAD = 1, F_LOGITS = 2, F_ACCEPT = 4, F_ADVANCE = 8, F_NOEMBED = 16 };   // NOEMBED: x rows are already in place

// `only` selects kernel classes (the benchmark times them in isolation); the default runs everything.
// C_FUSED: a class-restricted pass keeps the epilogue variants of the full step (the o / down / PLE projections that leave
// complete rows and the partial sums of the norms that follow them) instead of the plain ones.
enum { C_QKV = 1, C_O = 2, C_GATEUP = 4, C_DOWN = 8, C_HEAD = 16, C_PLE = 32, C_NORM = 64, C_ATTN = 256, C_MISC = 512,
       C_ALL = 1023, C_FUSED = 1024 };

// A model family beside the block-quantised one: how its weights are loaded, how its cache is laid out, and what a forward
// enqueues.  Sessions, round state, graphs, acceptance, sampling hooks and the exported API are the engine's own and the same
// for every family.
struct LgFamily {
    const char *name;
    void (*load)(Engine *e);                                       // weights + activations (e->m, e->ctx, e->stream are set)
    void (*release)(Engine *e);
    int  (*kv_slots)(const struct model *m);                       // cache entries (a layer that runs several times has one per run)
    int  (*kv_init)(struct kvcache *kv, const struct model *m, bool f32);   // fills kv_dim / seq / f16 and allocates; 0 / -1
    void (*bind)(Engine *e, const struct kvcache *kv);             // scratch that depends on the cache's geometry
    // M <= LG_MAXM rows at st->pos from st->toks (captured into graphs); with F_HEAD: e->hidden, argmax candidates in
    // e->amax_*, with F_LOGITS e->logits.  Returns the number of candidates per row.
    int  (*forward)(Engine *e, const struct kvcache *kv, int M, int flags, int only);
    void (*embed)(Engine *e, int M);                               // token embeddings of st->toks into e->x
    // The wide prompt pass: fills the cache rows of n tokens; logits of the n_want places listed (ascending) go to `logits`
    // (host, [n_want][n_vocab]).  Returns the number of tokens it took (the rest goes through `forward`).
    int  (*prefill)(Engine *e, const struct kvcache *kv, const int *toks, int n, int pos0, const int *want, int n_want, float *logits);
    int  (*bench_block)(Engine *e, const struct kvcache *kv, int n, int pos0, int only);   // kernels of one wide block, timing only
    // Told before n tokens run at pos (wide: as a prompt block; n < 0: rounds that only the device follows); false: the cache holds no state
    // for that position.
    bool (*start)(Engine *e, const struct kvcache *kv, int pos, int n, bool wide);
    bool (*prefix)(struct kvcache *kv, int n, bool restore, cudaStream_t s);               // what a saved prefix needs besides cache rows
};

struct WMat {
    uint4 *wq = nullptr; uint2 *ws = nullptr; uint2 *wd = nullptr; uint4 *wm = nullptr;      // tiles, scales (see lg_kernels.cuh)
    int fmt = 0, m = 0, k = 0, nkp = 0, n_row_tiles = 0, ldo = 0;
    size_t file_bytes = 0;
};

struct Panel { LgPanel p{}; };

struct LayerW {
    WMat qkv, o, gateup, down, inp_gate, proj;
    // q / k / v tensors of different formats cannot share one stacked matrix: they are kept apart, each multiplied on its
    // own into its rows of the projection buffer (qkv then only carries the row stride)
    std::vector<WMat> qkv_parts; std::vector<int> qkv_row0;
    float *attn_norm = nullptr, *q_norm = nullptr, *k_norm = nullptr, *post_attn = nullptr, *ffn_norm = nullptr,
          *post_ffw = nullptr, *post_norm = nullptr;
    float out_scale = 1.0f;
    int has_v = 1, owns_kv = 1, src = 0, local = 0, hd = 0, nkv = 0, nff = 0;
};

struct DraftBlockW {
    WMat q, o, gateup, down;
    float *attn_norm, *q_norm, *post_attn, *ffn_norm, *post_ffw;
    float out_scale; int hd, local, src;
};
struct DraftW {
    WMat pre, post, head;
    float *out_norm = nullptr;
    std::vector<DraftBlockW> blk;
    int ni = 0, nb = 0, nff = 0, n_head = 0, n_vocab = 0, has_post = 0;
    float eps = 0, base_full = 0, base_swa = 0, softcap = 0;
    // activations (one token)
    float *cat = nullptr, *x = nullptr, *hbuf = nullptr, *qbuf = nullptr, *qrot = nullptr, *obuf = nullptr, *gu = nullptr, *part = nullptr;
    float *amax_val = nullptr; int *amax_idx = nullptr, *best = nullptr;
    float *amax_val2 = nullptr, *margin = nullptr;      // runner-up logits per CTA; best - second best of the latest draft
    float2 *part_ml = nullptr;
    LgPanel p_cat{}, p_ni{}, p_attn{}, p_ff{};
    float2 *rope_local = nullptr, *rope_global = nullptr; int hd_local = 0, hd_global = 0;
    int n_slots_local = 0, n_slots_global = 0;
    std::map<std::string, cudaGraphExec_t> graphs;
};

// Buffers of the wide prompt pass (blocks of up to LG_PF_MAXN tokens), allocated at its first use.
struct PrefillBuf {
    bool ready = false;
    __half *a_ne = nullptr, *a_attn = nullptr, *a_ff = nullptr;     // f16 matmul inputs [LG_PF_MAXN][k]
    float *x = nullptr, *qkv = nullptr, *o = nullptr;               // residual rows, projection rows, o/down rows
    int *toks = nullptr, *pos = nullptr;                            // token ids; pos[g] = position of the g-th group of 8
    float2 *rope_local = nullptr, *rope_global = nullptr;
    __half *q_hi = nullptr, *q_lo = nullptr;                        // normed + rotated queries [LG_PF_MAXN][H][hd], f16 hi + lo
    float *tokrow = nullptr, *pproj = nullptr, *ipl = nullptr, *pg = nullptr;   // per-layer-embedding rows [LG_PF_MAXN][ple * n_layer], gate rows
    __half *a_ple = nullptr;
    float *rows = nullptr; int *ridx = nullptr;                     // media rows of the block and, per token, its row or -1
    int ld_attn = 0, ld_ff = 0;
};

struct Engine {
    const struct model *m = nullptr;
    const struct gguf_context *ctx = nullptr;
    cudaStream_t stream = nullptr;
    int sm_count = 148;
    // weights
    const LgFamily *fam = nullptr;            // set for a model that is not block-quantised; plan: that family's own state
    PlanModel *plan = nullptr;
    bool f32 = false;                         // plan models: every product and the cache in 32-bit
    std::vector<LayerW> L;
    WMat head, pmp;                           // token_embd (tied head), per_layer_model_proj
    uint8_t *ple_table = nullptr; int ple_table_type = 0;   // per_layer_token_embd, file layout
    float *out_norm = nullptr, *ple_proj_norm = nullptr, *rope_div = nullptr;
    float2 *rope_local = nullptr, *rope_global = nullptr; int hd_local = 0, hd_global = 0;
    int has_ple = 0;
    size_t weight_bytes = 0;
    // activations
    float *x = nullptr, *qkv = nullptr, *qrot = nullptr, *oout = nullptr, *gu = nullptr, *dout = nullptr, *hidden = nullptr,
          *h_prev = nullptr, *part = nullptr, *tokrow = nullptr, *pproj = nullptr, *ipl = nullptr, *pg = nullptr, *logits = nullptr;
    float *amax_val = nullptr; int *amax_idx = nullptr;
    float2 *part_ml = nullptr;
    LgPanel p_ne{}, p_attn{}, p_ff{}, p_ple{};
    int max_ks = 4, head_ctas = 0;
    int part_slots = 0;
    // session
    LgRoundState *st = nullptr;               // device
    LgRoundState *st_host = nullptr;          // pinned mirror for uploads / downloads
    int *log = nullptr, *replay = nullptr, *d_n_replay = nullptr; int n_replay = 0, replay_cap = 0;   // replay table (capacity grows; its length lives on the device)
    int *err = nullptr, *tickets = nullptr;
    std::map<std::string, cudaGraphExec_t> graphs;
    const struct kvcache *kv_bound = nullptr;
    DraftW *draft = nullptr; const struct mtp *draft_owner = nullptr;
    float *pick_rows = nullptr;               // host logits rows for model_pick
    long long launches = 0;                   // kernels enqueued by the most recent graph build
    int pdl = 1;                              // programmatic dependent launch (LG_PDL=0 turns it off)
    long long round_launches = 0;
    PrefillBuf pf;
    float4 *sums = nullptr;                   // SUMS epilogue: per work item and token the partial sums the next kernel builds the norms from
    int pos_hi = 0;                           // host-side upper bound of the device position (device-resident rounds)
    // One host synchronisation per round behind the blocking calls: mtp_draft_device runs the WHOLE round and keeps its
    // outcome here; the chained-draft and verify calls that follow are answered from it when they ask what was computed.
    struct { bool valid = false; int n = 0, pos = 0, adv = 0, toks[LG_MAXM] = {0}, out[LG_MAXM] = {0}; bool chained = false; } lazy;
    int replay_off = 0; bool lazy_replay = false;   // replay table index of a draft = its position + replay_off (lg_set_replay_origin)
    long long host_syncs = 0;                 // blocking device-to-host waits made by the reference-shaped calls
    float *d_margin_thr = nullptr;            // confidence margin below which a draft calls off the drafts after it (0: never)
    cudaEvent_t mid_event = nullptr;          // LG_MTP_PROFILE: recorded between the layers and the head of a forward
    int mm_launches = 0;                      // kernels in the captured matmul-only pass             // kernels in one captured round (lg_rounds_enqueue)
};

// Kernel launch on the engine's stream, marked for programmatic dependent launch so the kernel may
// start while its predecessor drains (every forward kernel begins with pdl_wait()).
template <typename... KArgs, typename... Args>
void launch_k(Engine *e, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = e->stream;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at; cfg.numAttrs = e->pdl ? 1 : 0;
    LG_CHECK(cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...));
    e->launches++;
}
// The same with the CTAs of one blockIdx.x forming a thread-block cluster (1, grid.y, 1).
template <typename... KArgs, typename... Args>
void launch_k_cluster_y(Engine *e, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = e->stream;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = 1; at[0].val.clusterDim.y = grid.y; at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at; cfg.numAttrs = e->pdl ? 2 : 1;
    LG_CHECK(cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...));
    e->launches++;
}


// Zero-filled device allocation.  The fill runs on the legacy stream, which does not order against the
// engine's non-blocking stream, so wait for it before anyone can use the buffer.
template <typename T> T *dalloc(size_t n) {
    T *p = nullptr;
    LG_CHECK(cudaMalloc(&p, n * sizeof(T) > 0 ? n * sizeof(T) : 16));
    LG_CHECK(cudaMemset(p, 0, n * sizeof(T)));
    LG_CHECK(cudaDeviceSynchronize());
    return p;
}

// Host -> device copy that is complete on return.  A pageable-source cudaMemcpy may return while
// its last DMA is still in flight on the legacy stream, which the engine's non-blocking stream does
// not order against, so wait for the device.
inline void h2d_sync(void *dst, const void *src, size_t bytes) {
    LG_CHECK(cudaMemcpy(dst, src, bytes, cudaMemcpyHostToDevice));
    LG_CHECK(cudaDeviceSynchronize());
}

inline float *upload_f32(const float *src, size_t n) {
    float *d = dalloc<float>(n);
    h2d_sync(d, src, n * 4);
    return d;
}

inline const struct gguf_tensor *find_t(const struct gguf_context *g, int L, const char *leaf) {
    char name[96];
    if (L >= 0) snprintf(name, sizeof name, "blk.%d.%s", L, leaf); else snprintf(name, sizeof name, "%s", leaf);
    return gguf_find_tensor(g, name);
}
inline int env_int(const char *name, int fb) { const char *v = getenv(name); return v && v[0] ? atoi(v) : fb; }

// Descriptor of a row-major matrix [rows][cols] for tiled copies: boxes of box_c columns (one 128-byte swizzle row) x box_r rows.
typedef CUresult (*EncodeTiledFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *,
                                  const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
inline CUtensorMap tiled_map(const void *ptr, CUtensorMapDataType type, long long cols, long long rows, long long row_bytes, int box_c, int box_r) {
    static EncodeTiledFn fn = nullptr;
    if (!fn) {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult qr;
        LG_CHECK(cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &qr));
        if (!p || qr != cudaDriverEntryPointSuccess) { fprintf(stderr, "lg_b200: the driver has no cuTensorMapEncodeTiled\n"); exit(1); }
        fn = (EncodeTiledFn)p;
    }
    CUtensorMap map;
    cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    cuuint64_t strides[1] = {(cuuint64_t)row_bytes};
    cuuint32_t box[2] = {(cuuint32_t)box_c, (cuuint32_t)box_r};
    cuuint32_t estr[2] = {1, 1};
    CUresult r = fn(&map, type, 2, (void *)ptr, dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                    CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) { fprintf(stderr, "lg_b200: cuTensorMapEncodeTiled failed (%d) for %lld x %lld\n", (int)r, rows, cols); exit(1); }
    return map;
}

void check_err(Engine *e);                    // waits for the stream; ends the process when a kernel raised the status word

}  // namespace lg

// The family that runs the model in `ctx`, or NULL for the block-quantised models.  Weak: a host that links the engine object
// alone has only those.
extern "C" const lg::LgFamily *lg_family_for(const struct gguf_context *ctx) __attribute__((weak));

#endif  // LG_ENGINE_H
