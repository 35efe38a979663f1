// lg_device.cuh -- device-side helpers and types shared by every kernel family of the library: warp / block sums,
// programmatic dependent launch, mbarriers with bounded waits, bulk and tiled copies, cluster exchange, ldmatrix / mma,
// tcgen05 issue and read-back, and the device-resident round state.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>
#include <cuda_fp16.h>
#include <stdint.h>

#define LG_MAXM 8              // widest verify block
#define LG_QMAX 32639.0f       // 127*256 + 127: keeps both bytes of the split in [-128,127]
#define LG_SPIN_LIMIT (1 << 20)

// error bits a kernel may raise in the engine's status word
#define LG_ERR_MBAR_TIMEOUT 1
#define LG_ERR_SEQ_POS 256       // a block at a position whose sequence state is gone

struct LgPanel {               // quantised activations of <= 8 tokens, k = 32*nsb columns
    int8_t *q;                 // [2][nsb][256]
    float2 *s;                 // [2][nsb][4]   (scale, scale * sum of the group's integers)
    int nsb;
};

// ---------------------------------------------------------------------------------------------
// small helpers
// ---------------------------------------------------------------------------------------------
__device__ __forceinline__ float warp_sum(float v) {
    #pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
    #pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
// Sum over the block in a fixed order (independent of anything but blockDim). `red` >= 32 floats.
__device__ __forceinline__ float block_sum(float v, float *red) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    int nw = (blockDim.x + 31) >> 5;
    float t = (threadIdx.x < nw) ? red[threadIdx.x] : 0.0f;
    if (threadIdx.x < 32) t = warp_sum(t);
    if (threadIdx.x == 0) red[0] = t;
    __syncthreads();
    return red[0];
}

__device__ __forceinline__ float gelu_tanh(float x) {
    return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
}

// Programmatic dependent launch: every kernel of a forward may be started before its predecessor
// has finished.  pdl_launch() lets the successor begin its own prologue; pdl_wait() blocks until the
// predecessor grid has completed and its writes are visible.  Nothing produced by an earlier kernel
// may be read, and nothing may be written, before pdl_wait().  (No-ops for a plain launch.)
__device__ __forceinline__ void pdl_launch() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

__device__ __forceinline__ uint32_t smem_u32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }

// ---- phase time stamps (profiling builds only: -DLG_STAMPS) ------------------------------------
// Thread 0 of a CTA records the global nanosecond timer at named points of a kernel into
// lg_stamps[launch tag][CTA][slot]; the host reads the array back after a forward and lays the launches of a
// layer on one time axis (lg_debug_stamps).  Compiled out of the product build.
#define LG_STAMP_LAUNCHES 96
#define LG_STAMP_CTAS 320
#define LG_STAMP_SLOTS 12
#ifdef LG_STAMPS
__device__ long long lg_stamps[LG_STAMP_LAUNCHES][LG_STAMP_CTAS][LG_STAMP_SLOTS];
__device__ __forceinline__ void lg_stamp(int tag, int slot) {
    if (threadIdx.x == 0 && tag >= 0 && tag < LG_STAMP_LAUNCHES) {
        const int cta = blockIdx.x + gridDim.x * (blockIdx.y + gridDim.y * blockIdx.z);
        if (cta < LG_STAMP_CTAS) {
            long long t;
            asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
            lg_stamps[tag][cta][slot] = t;
        }
    }
}
#define LG_STAMP(tag, slot) lg_stamp(tag, slot)
// the last slot of CTA 0 names the kernel (1 matmul store, 2 head, 3 GeGLU, 4 matmul with sums, 5 attention/ticket, 6 attention/cluster, 7 norm / residual update)
#define LG_STAMP_KIND(tag, kind) do { if (threadIdx.x == 0 && blockIdx.x == 0 && blockIdx.y == 0 && (tag) >= 0 && (tag) < LG_STAMP_LAUNCHES) lg_stamps[tag][0][LG_STAMP_SLOTS - 1] = (kind); } while (0)
#else
#define LG_STAMP(tag, slot) do { } while (0)
#define LG_STAMP_KIND(tag, kind) do { } while (0)
#endif

// streaming 16-byte weight load: read-only path, do not keep in L1
__device__ __forceinline__ uint4 ldg_stream16(const uint4 *p) {
    uint4 v;
    asm("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ void mbar_init(uint64_t *bar, int count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" :: "r"(smem_u32(bar)), "r"(count));
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t *bar, uint32_t bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" :: "r"(smem_u32(bar)), "r"(bytes) : "memory");
}
// dst, src 16-byte aligned, bytes a multiple of 16
__device__ __forceinline__ void bulk_g2s(void *dst, const void *src, uint32_t bytes, uint64_t *bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 :: "r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
// Bounded wait: returns false (and the caller raises LG_ERR_MBAR_TIMEOUT) instead of spinning forever.
__device__ __forceinline__ bool mbar_wait(uint64_t *bar, uint32_t parity) {
    for (int it = 0; it < LG_SPIN_LIMIT; ++it) {
        uint32_t ok;
        asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                     : "=r"(ok) : "r"(smem_u32(bar)), "r"(parity) : "memory");
        if (ok) return true;
    }
    return false;
}

__device__ __forceinline__ uint32_t cluster_rank() { uint32_t r; asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ void dsmem_store(float *local_addr, uint32_t rank, float v) {
    uint32_t la = smem_u32(local_addr), ra;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ra) : "r"(la), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" :: "r"(ra), "f"(v) : "memory");
}
// One f32 into a peer CTA's shared memory, counted (4 bytes) on that peer's mbarrier: the receiver waits for the byte
// count instead of a cluster-wide barrier, so threads that never join a barrier (a producer warp) are no obstacle.
__device__ __forceinline__ void dsmem_st_async_f32(float *local_addr, uint64_t *local_bar, uint32_t rank, float v) {
    uint32_t ra, rb;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ra) : "r"(smem_u32(local_addr)), "r"(rank));
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(rb) : "r"(smem_u32(local_bar)), "r"(rank));
    asm volatile("st.async.weak.shared::cluster.mbarrier::complete_tx::bytes.f32 [%0], %1, [%2];" :: "r"(ra), "f"(v), "r"(rb) : "memory");
}
// Bounded wait with cluster-scope acquire: the data counted on the barrier came from peer CTAs.
__device__ __forceinline__ bool mbar_wait_cluster(uint64_t *bar, uint32_t parity) {
    for (int it = 0; it < LG_SPIN_LIMIT; ++it) {
        uint32_t ok;
        asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                     : "=r"(ok) : "r"(smem_u32(bar)), "r"(parity) : "memory");
        if (ok) return true;
    }
    return false;
}

__device__ __forceinline__ void mbar_arrive(uint64_t *bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" :: "r"(smem_u32(bar)) : "memory");
}

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void *p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], const void *p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_f16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(void *dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

struct LgRoundState {          // lives in device memory; one per session
    int pos;                   // position of toks[0] of the round being built
    int toks[LG_MAXM];         // toks[0] = chosen token, toks[1..] = drafts
    int out[LG_MAXM];          // greedy successors of toks[j]
    int adv;                   // tokens advanced by the last verify (1..M)
    int n_emitted;             // tokens appended to the log so far
    int n_draft, n_accept;
    int dpos;                  // position the draft head is drafting for
    int stop;                  // this round's remaining drafts are called off (a draft's confidence margin fell below the threshold)
    int n_skipped;             // drafts called off so far
};

// ---- tiled copies and tcgen05 ------------------------------------------------------------------
// mbar_wait on a shared-space address that is already in a register
__device__ __forceinline__ bool mbar_wait_u32(uint32_t bar, uint32_t parity) {
    for (int it = 0; it < LG_SPIN_LIMIT; ++it) {
        uint32_t ok;
        asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                     : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
        if (ok) return true;
    }
    return false;
}

__device__ __forceinline__ void tma_load_2d(void *dst, const CUtensorMap *map, int x, int y, uint64_t *bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                 :: "r"(smem_u32(dst)), "l"(map), "r"(x), "r"(y), "r"(smem_u32(bar)) : "memory");
}
// K-major operand, 128-byte swizzle: rows of 128 bytes, 8-row groups 1024 bytes apart
__device__ __forceinline__ uint64_t umma_desc_k128(uint32_t saddr) {
    return (uint64_t)((saddr & 0x3FFFFu) >> 4) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void umma_f16(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
                 :: "r"(d_tmem), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate) : "memory");
}
__device__ __forceinline__ void umma_commit(uint64_t *bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" :: "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&r)[32]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x32.b32 "
                 "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
                   "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]),
                   "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]),
                   "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
                 : "r"(taddr) : "memory");
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}
