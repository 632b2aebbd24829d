// bf16 GEMM family on tcgen05 tensor cores: Y[t, n] = sum_k X[t, k] * W[n, k]  (+ epilogue)
//
// One kernel template covers every dense projection of the model, the per-head absorbed-MLA
// products and the routed-expert grouped GEMMs (reference ops: aclnnMm/BatchMatMul
// ggml/src/ggml-cann/aclnn_ops.cpp:4647-4693, aclnnGroupedMatmulV4 x3 + Silu + Mul 2258-2421).
//
// Design (swap-AB, weight-stationary M):
//  * the 128-row MMA "M" dimension is a tile of OUTPUT FEATURES (rows of W, K-major as stored), the
//    MMA "N" dimension is a tile of BN tokens (16..256).  Decode batches of 1..64 tokens therefore use
//    full 128-lane tensor-core instructions and stream each weight byte exactly once;
//  * operands are staged by TMA (128-byte swizzle, no multicast) into a ring of STAGES shared-memory
//    slots guarded by full/empty mbarriers; one elected thread issues tcgen05.mma into a TMEM
//    accumulator; four epilogue warps read it back with tcgen05.ld;
//  * split-K: when N/128 tiles cannot fill 148 SMs, the K range is split over several CTAs that write
//    fp32 partials to a scratch buffer; the last CTA to arrive (per-tile counter) reduces them and runs
//    the epilogue, then resets the counter so the buffers need no clearing between launches;
//  * DUAL mode keeps two accumulators (gate and up projections of the same tile) and stores
//    act(gate) * up — the gated-FFN epilogue — so the 2x wider intermediate never reaches HBM;
//  * grouped mode: blockIdx.z selects an expert; the token rows of that expert are a segment
//    [seg[e], seg[e+1]) of an expert-sorted activation matrix; segment bounds are read on the device
//    (no host sync, unlike aclnn_ops.cpp:2136-2146).
//  * every mbarrier wait is bounded; on expiry a status word is set and the CTA leaves normally.
#include "sm100.cuh"

#include <mutex>
#include <unordered_map>
#include <vector>
#include <string.h>

#include "comm_fused.cuh"
#include "jib_kernels.h"
#include "pdl.cuh"

using namespace sm100;

namespace {

constexpr int BM = 128;      // output features per CTA (MMA M)
constexpr int BK = 64;       // K elements per stage (128 bytes of bf16 = one swizzle row)
constexpr int UMMA_K = 16;
constexpr int NUM_THREADS = 192;   // warp0 TMA, warp1 MMA + TMEM owner, warps 2..5 epilogue

struct GemmArgs {
    void * out;
    const void * residual;
    const int * seg;          // grouped: expert segment offsets [batch+1] into the sorted rows, else null
    float * scratch;
    int * counters;
    int * status;
    long long ldo, out_batch_stride, ldr, res_batch_stride;
    int T, N, K;
    int splits, kb_per_split;
    int out_f32, res_f32;
    long long rows_total;     // rows of out (all batches of a grouped launch share them); stores beyond are refused
    long long scratch_elems;
    JibArCtx ar;              // peer-memory all-reduce fused into the epilogue (ar_on != 0)
    int ar_on, ar_site;
    int cluster_split;        // 1: the `splits` CTAs of a tile form a thread-block cluster and reduce through DSMEM
    // all-gather fused into the activation loads: rows of source rank s are complete once ag_flags[s] == *ag_epoch
    const unsigned * ag_flags;
    const unsigned * ag_epoch;
    int ag_rows, ag_world;    // rows per source rank, number of ranks
    unsigned ag_spin_limit;   // polls of the wait for a source's rows (0 = JIB_AR_SPIN_LIMIT)
    int ar_rs_rows;           // two-shot: > 0 delivers each reduced row only to rank row / ar_rs_rows (reduce-scatter)
    void * const * row_ptr;   // null, or per output row the address of its bf16 row (rows scattered to other buffers,
                              // possibly on other GPUs: the expert-parallel return path)
    const int * expert_list;  // grouped: null, or the experts the grid's z slots stand for (device; -1 = unused slot)
    int list_tiles;           // the list holds (token tile << 16 | expert) entries and gridDim.y is 1
    int pdl_flags;            // grouped pairs: bit 0 = release dependents after the own wait, bit 1 = segment table valid at start
    int w_evict_first;        // weight tiles are loaded with the L2 evict_first policy (each is read once: small batches)
    int act;                  // of a gated pair (JIB_ACT_*)
    int unary;                // of a single product (JIB_UNARY_*)
    float scale, softcap, cap2;      // cap2 = 2 scale / softcap
    const float * row_scale;  // JIB_UNARY_GELU: null, or a factor of every result row's product
    const float * bias;       // null, or [N]: a residual row that all rows share (then residual is null)
    int vec_store;            // bf16 result rows are written as 16-byte vectors through a shared-memory transpose
    const int * src_token;    // grouped, decode batches: x holds the T token rows unsorted, every expert multiplies all of
                              // them (one token tile) and sorted row i of the result is accumulator column src_token[i]
};

template <int BN, bool DUAL>
struct Cfg {
    static constexpr int A_BYTES = BM * BK * 2;
    static constexpr int B_BYTES = BN * BK * 2;
    static constexpr int STAGE_BYTES = (DUAL ? 2 : 1) * A_BYTES + B_BYTES;
    // Narrow token tiles are bandwidth-bound streams of small CTAs: give each half of the shared memory so
    // that two CTAs share an SM and one's prologue/epilogue hides behind the other's loads.
    static constexpr int SMEM_BUDGET = BN <= 32 ? 108 * 1024 : 200 * 1024;
    static constexpr int STAGES_RAW = SMEM_BUDGET / STAGE_BYTES;
    static constexpr int STAGES = STAGES_RAW > 8 ? 8 : STAGES_RAW;
    static constexpr int ACC_COLS = BN * (DUAL ? 2 : 1);
    static constexpr int TMEM_COLS = ACC_COLS <= 32 ? 32 : ACC_COLS <= 64 ? 64 : ACC_COLS <= 128 ? 128 : ACC_COLS <= 256 ? 256 : 512;
    static constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + 1024 /*align*/ + 256 /*barriers*/;
};

// Reduction side of the fused all-reduce for one tile (rows [t_begin, t_end) x 128 features starting at n0), run by the
// 128 epilogue threads.  The partials sit in global memory (`slots`: world slots of stride `slot_stride` floats), so the
// mapping is free: a thread owns 4 adjacent features (one 16-byte load per slot) of every 4th row, and 4 rows are kept
// in flight at once -- world x 4 independent loads per thread instead of a serial chain per row.  The sum runs in rank
// order.  `store(row, n, float4)` receives each finished quad.
template <typename Store>
__device__ __forceinline__ void ar_reduce_tile(const float * slots, size_t slot_stride, int world, int d_max, long long row_base,
                                               int t_begin, int t_end, int n0, int N, const void * residual, int res_f32, long long rbase,
                                               long long ldr, int ltid, Store store) {
    const int fq = (ltid & 31) * 4, rsub = ltid >> 5;
    const int n = n0 + fq;
    if (n >= N) return;
    for (int t0 = t_begin + rsub; t0 < t_end; t0 += 16) {
        float4 acc[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) acc[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s = 0; s < world; ++s) {
            float4 v[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int t = t0 + 4 * u;
                v[u] = t < t_end ? __ldcg((const float4 *) (slots + (size_t) s * slot_stride + (size_t) (row_base + t) * d_max + n))
                                 : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int u = 0; u < 4; ++u) { acc[u].x += v[u].x; acc[u].y += v[u].y; acc[u].z += v[u].z; acc[u].w += v[u].w; }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int t = t0 + 4 * u;
            if (t >= t_end) break;
            const long long row = row_base + t;
            if (residual != nullptr) {
                const long long ri = rbase + row * ldr + n;
                if (res_f32) {
                    const float4 rv = *(const float4 *) ((const float *) residual + ri);
                    acc[u].x += rv.x; acc[u].y += rv.y; acc[u].z += rv.z; acc[u].w += rv.w;
                } else {
                    const uint2 raw = *(const uint2 *) ((const __nv_bfloat16 *) residual + ri);
                    const float2 a = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.x);
                    const float2 b = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.y);
                    acc[u].x += a.x; acc[u].y += a.y; acc[u].z += b.x; acc[u].w += b.y;
                }
            }
            store(row, n, acc[u]);
        }
    }
}

__device__ __forceinline__ uint2 pack_bf16x4(float4 v) {
    uint2 o;
    *(__nv_bfloat162 *) &o.x = __floats2bfloat162_rn(v.x, v.y);
    *(__nv_bfloat162 *) &o.y = __floats2bfloat162_rn(v.z, v.w);
    return o;
}

// act(z) = z * sigmoid(z), or for the tanh form of gelu z * sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3)): 0.5 (1 + tanh(u)) = sigmoid(2 u)
__device__ __forceinline__ float gated(float x, int act) {
    const float z = act == JIB_ACT_GELU_TANH ? 1.5957691216057308f * (x + 0.044715f * x * x * x) : x;
    return x / (1.0f + __expf(-z));
}

// JIB_UNARY_* of a single product (FN instances: the plain kernels stay free of it); softcap y = c tanh(s v / c) with tanh(u) = 1 - 2 / (1 + e^{2u})
__device__ __forceinline__ float unary(float v, const GemmArgs & a) {
    if (a.unary == JIB_UNARY_RELU2) return v > 0.f ? v * v : 0.f;
    if (a.softcap <= 0.f) return v * a.scale;
    return a.softcap * (1.f - __fdividef(2.f, 1.f + __expf(fminf(v * a.cap2, 80.f))));
}
// FN instances: 0 the product itself, 1 relu^2 and softcap, 2 gelu of the product times its row's factor (a row past the tile's last has none),
// 3 the product plus its feature's bias (an epilogue thread holds one feature: a register).
// erfc(|z|) by Abramowitz and Stegun's formula 7.1.26 (absolute error 1.5e-7): a polynomial in 1 / (1 + p |z|) times e^{-z^2}.
__device__ __forceinline__ float gelu(float v) {
    const float z = fabsf(v) * 0.70710678118654752f;
    float t, e;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(t) : "f"(1.f + 0.3275911f * z));
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-1.4426950408889634f * z * z));
    const float p = t * (0.254829592f + t * (-0.284496736f + t * (1.421413741f + t * (-1.453152027f + t * 1.061405429f))));
    const float half = 0.5f * v * (p * e);                   // v erfc(|z|) / 2
    return v > 0.f ? v - half : half;
}
__device__ __forceinline__ float row_factor(const GemmArgs & a, long long row, bool valid) {
    return a.row_scale != nullptr && valid ? __ldg(a.row_scale + row) : 1.f;
}
// by: the row's factor (FN 2) or the feature's bias (FN 3)
template <int FN>
__device__ __forceinline__ float function_of(float v, const GemmArgs & a, float by) {
    if (FN == 0) return v;
    if (FN == 3) return v + by;
    if (FN == 1) return unary(v, a);
    return gelu(v * by);
}

// Cluster-wide barrier (all threads of all CTAs of the cluster) and a load from a peer CTA's shared memory.
__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ float ld_dsmem_f32(uint32_t local_smem_addr, uint32_t cta_rank) {
    uint32_t remote;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_smem_addr), "r"(cta_rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
    return v;
}

template <int BN, bool DUAL, int FN>
__global__ void __launch_bounds__(NUM_THREADS, 1)
gemm_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmA2,
            const __grid_constant__ CUtensorMap tmB, const GemmArgs args) {
    using C = Cfg<BN, DUAL>;
    extern __shared__ uint8_t smem_raw[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    const int n0 = blockIdx.x * BM;
    const int splits = args.splits;
    const int slot = blockIdx.z / splits;          // batch index, or (grouped with an expert list) position in that list
    const int split = blockIdx.z - slot * splits;
    int batch = slot;
    int row0 = blockIdx.y * BN;      // first token row of this tile, relative to the segment / matrix (list_tiles: from the list)
    int rows_valid = args.T;         // rows of this batch's matrix
    int row_base = 0;                // grouped: offset of the expert's segment in the sorted rows
    JIB_KS(1, 0);
    // Grouped launches need the segment table.  Normally the routing kernel just before produced it, so they wait first.
    // A pair of grouped launches (gate|up, then down) shares one table: the first of the pair (pdl_flags bit 0) releases its
    // dependents only AFTER its own wait, which tells the second (bit 1) that the table is complete when it starts -- it
    // reads the table and requests its weight tiles before waiting for the first launch's results.
    // The dependents are released further down, once this CTA holds its tensor-memory columns: tcgen05.alloc blocks until
    // columns are free, so a CTA of the NEXT grid that became resident early, took columns and then sat in its own
    // dependency wait could starve a CTA of THIS grid that had yet to start on that SM -- for good.  Released after the
    // allocation (a CTA that leaves early releases by leaving), the next grid starts only when every CTA of this one has
    // its columns.
    const bool seg_early = args.seg != nullptr && (args.pdl_flags & 2) != 0;
    if (args.seg != nullptr && !seg_early) pdl_wait();
    if (args.seg != nullptr) {
        // decode batches hit few of the experts: the grid then covers a list of the experts that have rows (written by the
        // sort next to the segment table, -1 past its end) instead of all of them
        if (args.expert_list != nullptr) {
            batch = args.expert_list[slot];
            if (args.list_tiles && batch >= 0) {       // entry = token tile << 16 | expert: the grid walks (expert, tile) pairs
                row0 = (batch >> 16) * BN;
                batch &= 0xffff;
            }
        }
        if (batch < 0) {
            rows_valid = 0;
        } else {
            row_base = args.seg[batch];
            rows_valid = args.seg[batch + 1] - row_base;
        }
    }
    if (row0 >= rows_valid) {        // whole CTA: nothing to do (empty expert / tail tile)
        if (seg_early) pdl_wait();
        return;
    }

    const int num_kb = (args.K + BK - 1) / BK;
    const int kb0 = split * args.kb_per_split;
    const int kb1 = min(num_kb, kb0 + args.kb_per_split);
    const int nkb = kb1 - kb0;

    // ---- shared memory carve-up ----
    uint8_t * tiles = (uint8_t *) (((uintptr_t) smem_raw + 1023) & ~(uintptr_t) 1023);
    uint64_t * bars = (uint64_t *) (tiles + C::STAGES * C::STAGE_BYTES);
    uint64_t * full = bars;
    uint64_t * empty = bars + C::STAGES;
    uint64_t * acc_ready = bars + 2 * C::STAGES;
    uint32_t * tmem_slot = (uint32_t *) (bars + 2 * C::STAGES + 1);
    int * flag = (int *) (tmem_slot + 1);

    if (threadIdx.x == 0) {
        for (int s = 0; s < C::STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        mbar_init(acc_ready, 1);
        fence_barrier_init();
        prefetch_tmap(&tmA);
        prefetch_tmap(&tmB);
        if (DUAL) prefetch_tmap(&tmA2);
        *flag = 0;
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, C::TMEM_COLS);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (args.seg != nullptr && (args.pdl_flags & 1) != 0) pdl_launch_dependents();      // first of a pair: always here
    else PDL_TRIGGER_TOP();
    const uint32_t tmem = *tmem_slot;
    // Everything above touched only shared/tensor memory and launch-invariant data; activations, the residual,
    // scratch and the output belong to the stream order from here on.
    const bool early = args.seg == nullptr || seg_early;     // other grouped launches waited above

    if (warp == 0) {
        // ================= TMA producer =================
        if (elect_one()) {
            const int a_z = batch;
            const int b_z = args.seg != nullptr ? 0 : batch;
            const int b_row = args.src_token != nullptr ? 0 : row_base + row0;
            // Weights are launch-invariant: their tiles of the first ring pass are requested BEFORE the wait for the
            // previous kernel, so the HBM latency of the stream's head overlaps that kernel's tail.  The activation
            // tile of each stage follows after the wait and completes the same barrier phase.
            const uint64_t wpol = l2_policy_evict_first();
            const bool wfirst = args.w_evict_first != 0;
            int pre = 0;
            if (early && args.ag_flags == nullptr) {
                pre = min(nkb, C::STAGES);
                for (int i = 0; i < pre; ++i) {
                    uint8_t * st = tiles + i * C::STAGE_BYTES;
                    mbar_expect_tx(&full[i], C::STAGE_BYTES);
                    const int k = (kb0 + i) * BK;
                    if (wfirst) {
                        tma_load_3d_hint(st, &tmA, &full[i], k, n0, a_z, wpol);
                        if (DUAL) tma_load_3d_hint(st + C::A_BYTES, &tmA2, &full[i], k, n0, a_z, wpol);
                    } else {
                        tma_load_3d(st, &tmA, &full[i], k, n0, a_z);
                        if (DUAL) tma_load_3d(st + C::A_BYTES, &tmA2, &full[i], k, n0, a_z);
                    }
                }
            }
            if (early) pdl_wait();
            JIB_KS_ANY(1, 1);
            if (args.ag_flags != nullptr) {
                // the token rows of this tile were pushed by other ranks: wait (bounded) for the sources that cover
                // them, then order the peers' generic-proxy stores before this thread's async-proxy (TMA) reads
                const unsigned want = *args.ag_epoch;
                const int lo = (int) ((row_base + row0) / args.ag_rows);
                const int hi = min((int) ((row_base + row0 + BN - 1) / args.ag_rows), args.ag_world - 1);
                for (int src = lo; src <= hi; ++src) {
                    bool got = false;
                    for (unsigned it = 0, lim = args.ag_spin_limit != 0 ? args.ag_spin_limit : JIB_AR_SPIN_LIMIT; it < lim; ++it) {
                        if (jib_ld_acquire_sys(args.ag_flags + src) == want) { got = true; break; }
                        __nanosleep(40);
                    }
                    if (!got) jib_report(args.status, JIB_ERR_WAIT_TIMEOUT, 6, src);
                }
                asm volatile("fence.proxy.async;" ::: "memory");
            }
            for (int i = 0; i < nkb; ++i) {
                const int s = i % C::STAGES;
                const uint32_t ph = (i / C::STAGES) & 1;
                uint8_t * st = tiles + s * C::STAGE_BYTES;
                const int k = (kb0 + i) * BK;
                if (i >= pre) {
                    if (!mbar_wait(&empty[s], ph ^ 1)) { jib_report(args.status, JIB_ERR_WAIT_TIMEOUT, 1, i); break; }
                    mbar_expect_tx(&full[s], C::STAGE_BYTES);
                    if (wfirst) {
                        tma_load_3d_hint(st, &tmA, &full[s], k, n0, a_z, wpol);
                        if (DUAL) tma_load_3d_hint(st + C::A_BYTES, &tmA2, &full[s], k, n0, a_z, wpol);
                    } else {
                        tma_load_3d(st, &tmA, &full[s], k, n0, a_z);
                        if (DUAL) tma_load_3d(st + C::A_BYTES, &tmA2, &full[s], k, n0, a_z);
                    }
                }
                tma_load_3d(st + (DUAL ? 2 : 1) * C::A_BYTES, &tmB, &full[s], k, b_row, b_z);
            }
            JIB_KS_ANY(1, 2);
            PDL_TRIGGER_LATE();      // every load of this CTA is in flight: the next kernel may start its own
        } else if (early) {
            pdl_wait();
        }
        __syncwarp();
        if (args.cluster_split) { cluster_sync_all(); cluster_sync_all(); }
    } else if (warp == 1) {
        // ================= MMA issuer =================
        if (early) pdl_wait();
        if (elect_one()) {
            constexpr uint32_t idesc = idesc_bf16(BM, BN);
            bool ok = true;
            for (int i = 0; i < nkb && ok; ++i) {
                const int s = i % C::STAGES;
                const uint32_t ph = (i / C::STAGES) & 1;
                if (!mbar_wait(&full[s], ph)) { jib_report(args.status, JIB_ERR_WAIT_TIMEOUT, 2, i); ok = false; break; }
                tc_fence_after();
                const uint32_t a_addr = smem_u32(tiles + s * C::STAGE_BYTES);
                const uint32_t b_addr = a_addr + (DUAL ? 2 : 1) * C::A_BYTES;
#pragma unroll
                for (int kk = 0; kk < BK / UMMA_K; ++kk) {
                    const uint64_t bd = desc_k_sw128(b_addr + kk * UMMA_K * 2);
                    mma_bf16(tmem, desc_k_sw128(a_addr + kk * UMMA_K * 2), bd, idesc, (i | kk) != 0);
                    if (DUAL)
                        mma_bf16(tmem + BN, desc_k_sw128(a_addr + C::A_BYTES + kk * UMMA_K * 2), bd, idesc, (i | kk) != 0);
                }
                mma_commit(&empty[s]);     // frees the slot once these MMAs have read it
            }
            mma_commit(acc_ready);         // accumulators complete (also arrives after a failed wait)
        }
        __syncwarp();
        if (args.cluster_split) { cluster_sync_all(); cluster_sync_all(); }
    } else {
        // ================= epilogue (warps 2..5) =================
        if (early) pdl_wait();
        const int q = warp & 3;                   // TMEM lane quarter this warp may access
        const int r = q * 32 + lane;              // feature row inside the tile
        const int n = n0 + r;
        const float bias = FN == 3 && n < args.N ? args.bias[n] : 0.f;
        const bool acc_ok = mbar_wait(acc_ready, 0);
        if (!acc_ok) jib_report(args.status, JIB_ERR_WAIT_TIMEOUT, 3, 0);
        tc_fence_after();
        JIB_KS_T(1, 4, 64);
        const uint32_t tbase = tmem + ((uint32_t) (q * 32) << 16);
        const int tile_id = (slot * gridDim.y + blockIdx.y) * gridDim.x + blockIdx.x;
        if (args.ar_on != 0 && (threadIdx.x & 127) == 0) JIB_TS(30, args.ar_site, tile_id, split);
        constexpr int ACC = DUAL ? 2 : 1;
        float * part = nullptr;
        bool do_final = true;

        const bool csplit = args.cluster_split != 0;
        const bool src_mode = args.src_token != nullptr;
        // accumulator columns that hold data: the tile's valid token rows, or (src mode) all T tokens
        const int ncols = src_mode ? min(BN, args.T) : min(BN, rows_valid - row0);
        float * stage = (float *) tiles;          // pipeline buffers are idle once the accumulators are complete
        const long long obase = (long long) batch * args.out_batch_stride;
        const long long rbase = (long long) batch * args.res_batch_stride;
        // fused all-reduce: the tile's fp32 values go to slot [rank] of every peer instead of `out`
        unsigned ar_epoch = 0;
        size_t ar_par = 0;
        int ar_owner = 0;
        size_t ar_opar = 0;           // two-shot: offset of this call site's half of the result buffer (elements)
        if (args.ar_on) {
            ar_epoch = *args.ar.epoch;
            const int par = (args.ar_site + (int) (ar_epoch % 2u) * (args.ar.n_sites & 1)) & 1;
            const int mr = args.ar_on == 2 ? args.ar.max_rows2 : args.ar.max_rows;
            ar_par = (size_t) par * ((size_t) args.ar.world * mr * args.ar.d_max);
            ar_opar = (size_t) par * ((size_t) mr * args.ar.d_max);
            ar_owner = tile_id % args.ar.world;
        }
        // One finished element: feature n of row (row_base + t_rel); gv / uv are the summed accumulators.
        auto finish = [&](int t_rel, float gv, float uv) {
            const long long row = row_base + t_rel;
            if (row >= args.rows_total) { jib_report(args.status, JIB_ERR_BOUNDS, 5, (int) row); return; }
            float y = DUAL ? gated(gv, args.act) * uv : function_of<FN>(gv, args, FN == 2 ? row_factor(args, row, true) : bias);
            if (args.ar_on == 2) {      // two-shot: the partial goes to the tile's owner only
                args.ar.recv2[ar_owner][ar_par + ((size_t) args.ar.rank * args.ar.max_rows2 + row) * args.ar.d_max + n] = y;
                return;
            }
            if (args.ar_on) {
                const size_t off = ar_par + ((size_t) args.ar.rank * args.ar.max_rows + row) * args.ar.d_max + n;
                for (int p = 0; p < args.ar.world; ++p) args.ar.recv[p][off] = y;
                return;
            }
            if (args.row_ptr != nullptr) {
                __nv_bfloat16 * dst = (__nv_bfloat16 *) __ldg((const unsigned long long *) args.row_ptr + row);
                if (dst != nullptr) dst[n] = __float2bfloat16(y);
                return;
            }
            if (args.residual != nullptr) {
                const long long ri = rbase + row * args.ldr + n;
                y += args.res_f32 ? ((const float *) args.residual)[ri] : __bfloat162float(((const __nv_bfloat16 *) args.residual)[ri]);
            }
            const long long oi = obase + row * args.ldo + n;
            if (args.out_f32) ((float *) args.out)[oi] = y;
            else ((__nv_bfloat16 *) args.out)[oi] = __float2bfloat16(y);
        };

        if (csplit) {
            // split-K inside a cluster: every CTA parks its fp32 partial in its own shared memory ([acc][BN tokens][128
            // features]).  Without a fused collective the reduction is spread over the cluster: CTA `split` sums token
            // columns split, split + splits, ... of all peers through DSMEM (in split order, so the sum does not depend on
            // who computes it) and finishes them -- splits x fewer remote loads per thread than one CTA reducing the
            // whole tile.  With a fused collective CTA 0 reduces the tile, because the exchange is signalled per tile.
            const bool spread = args.ar_on == 0;
            if ((split != 0 || spread) && acc_ok) {
#pragma unroll 1
                for (int a = 0; a < ACC; ++a)
#pragma unroll 1
                    for (int c = 0; c < BN; c += 16) {
                        if (c >= ncols) break;
                        uint32_t v[16];
                        tmem_ld16(tbase + a * BN + c, v);
                        tmem_ld_wait();
#pragma unroll
                        for (int j = 0; j < 16; ++j) stage[(a * BN + c + j) * BM + r] = __uint_as_float(v[j]);
                    }
            }
            cluster_sync_all();
            JIB_KS_T(1, 5, 64);
            do_final = split == 0 && !spread;
            if (spread) {
                const uint32_t sbase = smem_u32(stage);
                const int n_items = src_mode ? rows_valid : ncols;
#pragma unroll 1
                for (int it = split; it < n_items; it += splits) {
                    const int col = src_mode ? min(max(__ldg(args.src_token + row_base + it), 0), BN - 1) : it;
                    float gsum[8], usum[8];
#pragma unroll
                    for (int pr = 0; pr < 8; ++pr) {
                        gsum[pr] = pr < splits ? ld_dsmem_f32(sbase + (uint32_t) ((col * BM + r) * 4), pr) : 0.f;
                        if (DUAL) usum[pr] = pr < splits ? ld_dsmem_f32(sbase + (uint32_t) (((BN + col) * BM + r) * 4), pr) : 0.f;
                    }
                    float gv = 0.f, uv = 0.f;
#pragma unroll
                    for (int pr = 0; pr < 8; ++pr) { gv += gsum[pr]; if (DUAL) uv += usum[pr]; }
                    if (n < args.N) finish(src_mode ? it : row0 + it, gv, uv);
                }
            }
        }

        if (splits > 1 && !csplit) {
            // 1) publish this split's fp32 partial: layout [acc][BN tokens][128 features]
            part = args.scratch + ((size_t) tile_id * splits) * (ACC * BN * BM);
            float * mine = part + (size_t) split * (ACC * BN * BM);
            const bool in_scratch = ((long long) tile_id * splits + splits) * (ACC * BN * BM) <= args.scratch_elems;
            if (!in_scratch) jib_report(args.status, JIB_ERR_BOUNDS, 4, tile_id);
            if (acc_ok && in_scratch) {
#pragma unroll 1
                for (int a = 0; a < ACC; ++a)
#pragma unroll 1
                    for (int c = 0; c < BN; c += 16) {
                        if (c >= ncols) break;
                        uint32_t v[16];
                        tmem_ld16(tbase + a * BN + c, v);
                        tmem_ld_wait();
#pragma unroll
                        for (int j = 0; j < 16; ++j) mine[(size_t) (a * BN + c + j) * BM + r] = __uint_as_float(v[j]);
                    }
            }
            __threadfence();
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (threadIdx.x == 64) {
                const int old = atomicAdd(&args.counters[tile_id], 1);
                const int last = old == splits - 1;
                if (last) args.counters[tile_id] = 0;      // ready for the next launch
                *flag = last;
            }
            asm volatile("bar.sync 1, 128;" ::: "memory");
            do_final = *flag != 0;
            if (do_final) __threadfence();
            JIB_KS_T(1, 5, 64);
            if (do_final && !in_scratch) do_final = false;
        }

        if (do_final && acc_ok && src_mode) {
            // one sorted row at a time: its token's accumulator column (summed over the splits when there are several)
#pragma unroll 1
            for (int it = 0; it < rows_valid; ++it) {
                const int col = min(max(__ldg(args.src_token + row_base + it), 0), BN - 1);
                float gv = 0.f, uv = 0.f;
                if (splits > 1) {
                    for (int s = 0; s < splits; ++s) {
                        const float * p = part + (size_t) s * (ACC * BN * BM);
                        gv += __ldcg(p + (size_t) col * BM + r);
                        if (DUAL) uv += __ldcg(p + (size_t) (BN + col) * BM + r);
                    }
                } else {
                    gv = __uint_as_float(tmem_ld1(tbase + col));
                    if (DUAL) uv = __uint_as_float(tmem_ld1(tbase + BN + col));
                    tmem_ld_wait();
                }
                if (n < args.N) finish(it, gv, uv);
            }
        } else if (do_final && acc_ok) {
#pragma unroll 1
            for (int c = 0; c < BN; c += 16) {
                if (c >= ncols) break;
                float g[16], u[16];
                if (splits > 1 && !csplit) {
#pragma unroll
                    for (int j = 0; j < 16; ++j) { g[j] = 0.f; u[j] = 0.f; }
                    // only the valid token columns are summed; 4 splits per trip keep 4 x jn loads in flight
                    const int jn = min(16, ncols - c);
#pragma unroll 4
                    for (int s = 0; s < splits; ++s) {
                        const float * p = part + (size_t) s * (ACC * BN * BM);
#pragma unroll
                        for (int j = 0; j < 16; ++j) {
                            if (j < jn) {
                                g[j] += __ldcg(p + (size_t) (c + j) * BM + r);
                                if (DUAL) u[j] += __ldcg(p + (size_t) (BN + c + j) * BM + r);
                            }
                        }
                    }
                } else {
                    uint32_t v[16];
                    tmem_ld16(tbase + c, v);
                    tmem_ld_wait();
                    if (c == 0) JIB_KS_T(1, 7, 64);
#pragma unroll
                    for (int j = 0; j < 16; ++j) g[j] = __uint_as_float(v[j]);
                    if (DUAL) {
                        tmem_ld16(tbase + BN + c, v);
                        tmem_ld_wait();
#pragma unroll
                        for (int j = 0; j < 16; ++j) u[j] = __uint_as_float(v[j]);
                    }
                    if (csplit) {
                        const int jn = min(16, ncols - c);
                        const uint32_t sbase = smem_u32(stage);
                        for (int pr = 1; pr < splits; ++pr) {
#pragma unroll
                            for (int j = 0; j < 16; ++j) {
                                if (j < jn) {
                                    g[j] += ld_dsmem_f32(sbase + (uint32_t) (((c + j) * BM + r) * 4), pr);
                                    if (DUAL) u[j] += ld_dsmem_f32(sbase + (uint32_t) (((BN + c + j) * BM + r) * 4), pr);
                                }
                            }
                        }
                    }
                }
                if (args.vec_store) {
                    // The accumulators hold [feature lane][token column]; the result is [token][feature].  Transpose 16 token
                    // columns through shared memory (fp32, two buffers in the idle pipeline area) so that a thread stores 8
                    // adjacent features of one token row as one 16-byte vector (residual added in fp32 before rounding).
                    const int ltid = (int) threadIdx.x - 64;
                    float * sb = stage + ((c >> 4) & 1) * (16 * BM);
                    float by[FN == 2 ? 16 : 1];
                    if (FN == 2) {
#pragma unroll
                        for (int j = 0; j < 16; ++j) by[FN == 2 ? j : 0] = row_factor(args, (long long) row_base + row0 + c + j, c + j < ncols);
                    }
#pragma unroll
                    for (int j = 0; j < 16; ++j)
                        sb[j * BM + r] = DUAL ? gated(g[j], args.act) * u[j] : function_of<FN>(g[j], args, FN == 2 ? by[FN == 2 ? j : 0] : bias);
                    asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll 1
                    for (int it = 0; it < 2; ++it) {
                        const int tok = (ltid >> 4) + it * 8, fg = (ltid & 15) * 8;
                        const int col = c + tok, nn = n0 + fg;
                        if (col >= ncols || nn >= args.N) continue;
                        const long long row = row_base + row0 + col;
                        if (row >= args.rows_total) { jib_report(args.status, JIB_ERR_BOUNDS, 5, (int) row); continue; }
                        float4 a = *(const float4 *) (sb + tok * BM + fg), b = *(const float4 *) (sb + tok * BM + fg + 4);
                        if (args.ar_on) {
                            // fused all-reduce: the fp32 partial goes to slot [rank] of every peer (one-shot) or of the
                            // tile's owner (two-shot) as 16-byte stores; the residual is added after the reduction
                            if (args.ar_on == 2) {
                                float * dst = args.ar.recv2[ar_owner] + ar_par + ((size_t) args.ar.rank * args.ar.max_rows2 + row) * args.ar.d_max + nn;
                                *(float4 *) dst = a;
                                *(float4 *) (dst + 4) = b;
                            } else {
                                const size_t off = ar_par + ((size_t) args.ar.rank * args.ar.max_rows + row) * args.ar.d_max + nn;
                                for (int p = 0; p < args.ar.world; ++p) {
                                    *(float4 *) (args.ar.recv[p] + off) = a;
                                    *(float4 *) (args.ar.recv[p] + off + 4) = b;
                                }
                            }
                            continue;
                        }
                        if (args.residual != nullptr) {
                            const long long ri = rbase + row * args.ldr + nn;
                            if (args.res_f32) {
                                const float4 ra = *(const float4 *) ((const float *) args.residual + ri);
                                const float4 rb = *(const float4 *) ((const float *) args.residual + ri + 4);
                                a.x += ra.x; a.y += ra.y; a.z += ra.z; a.w += ra.w;
                                b.x += rb.x; b.y += rb.y; b.z += rb.z; b.w += rb.w;
                            } else {
                                const uint4 raw = *(const uint4 *) ((const __nv_bfloat16 *) args.residual + ri);
                                const float2 r0 = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.x);
                                const float2 r1 = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.y);
                                const float2 r2 = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.z);
                                const float2 r3 = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.w);
                                a.x += r0.x; a.y += r0.y; a.z += r1.x; a.w += r1.y;
                                b.x += r2.x; b.y += r2.y; b.z += r3.x; b.w += r3.y;
                            }
                        }
                        const uint2 lo = pack_bf16x4(a), hi = pack_bf16x4(b);
                        __nv_bfloat16 * dst = args.row_ptr != nullptr
                                                  ? (__nv_bfloat16 *) __ldg((const unsigned long long *) args.row_ptr + row)
                                                  : (__nv_bfloat16 *) args.out + obase + row * args.ldo;
                        if (dst != nullptr) *(uint4 *) (dst + nn) = make_uint4(lo.x, lo.y, hi.x, hi.y);
                    }
                } else if (n < args.N) {
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        if (c + j >= ncols) break;
                        finish(row0 + c + j, g[j], DUAL ? u[j] : 0.f);
                    }
                }
            }
        }
        JIB_KS_T(1, 8, 64);
        if (do_final && acc_ok) {
            if (args.ar_on == 2) {
                // signal the owner; the owner waits (bounded) for every source, sums the slots in rank order, adds the
                // residual and stores the bf16 tile into every rank's result buffer; everybody waits for that delivery
                const int ltid = (int) threadIdx.x - 64;
                const bool ok = jib_ar2_signal_owner(args.ar, args.ar_site, tile_id, ar_owner, ar_epoch, 128, ltid);
                if (args.ar.rank == ar_owner && ok) {
                    const int world = args.ar.world;
                    ar_reduce_tile(args.ar.recv2[args.ar.rank] + ar_par, (size_t) args.ar.max_rows2 * args.ar.d_max, world, args.ar.d_max,
                                   row_base, row0, min(rows_valid, row0 + BN), n0, args.N, args.residual, args.res_f32, rbase, args.ldr,
                                   ltid, [&](long long row, int nn, float4 v) {
                                       const uint2 o = pack_bf16x4(v);
                                       const size_t oi = ar_opar + (size_t) row * args.ar.d_max + nn;
                                       if (args.ar_rs_rows > 0) {       // reduce-scatter: the row's owner only
                                           const int p = min((int) (row / args.ar_rs_rows), world - 1);
                                           *(uint2 *) ((__nv_bfloat16 *) args.ar.out2[p] + oi) = o;
                                       } else {
                                           for (int p = 0; p < world; ++p) *(uint2 *) ((__nv_bfloat16 *) args.ar.out2[p] + oi) = o;
                                       }
                                   });
                }
                jib_ar2_deliver_and_wait(args.ar, args.ar_site, tile_id, ar_owner, ar_epoch, 128, ltid);
            } else if (args.ar_on) {
                // signal every peer, wait (bounded) for every source, then sum the slots in rank order
                jib_ar_signal_and_wait(args.ar, args.ar_site, tile_id, ar_epoch, 128, (int) threadIdx.x - 64);
                ar_reduce_tile(args.ar.recv[args.ar.rank] + ar_par, (size_t) args.ar.max_rows * args.ar.d_max, args.ar.world, args.ar.d_max,
                               row_base, row0, min(rows_valid, row0 + BN), n0, args.N, args.residual, args.res_f32, rbase, args.ldr,
                               (int) threadIdx.x - 64, [&](long long row, int nn, float4 v) {
                                   const long long oi = obase + row * args.ldo + nn;
                                   if (args.out_f32) *(float4 *) ((float *) args.out + oi) = v;
                                   else *(uint2 *) ((__nv_bfloat16 *) args.out + oi) = pack_bf16x4(v);
                               });
            }
        }
        JIB_KS_T(1, 6, 64);
        if (csplit) cluster_sync_all();           // peers keep their shared memory alive until CTA 0 has read it
    }

    // ---- teardown ----
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, C::TMEM_COLS);
    JIB_KS(1, 9);
}

// ---------------------------------------------------------------------------------------------
// Persistent form for launches with several waves of tiles (prompt chunks): one CTA per SM walks the tile list, the TMA
// ring keeps streaming across tile boundaries, and the accumulators are double-buffered in tensor memory, so the
// epilogue of tile i (tcgen05.ld, SiLU, transpose, 16-byte stores) runs under the MMAs of tile i + 1 instead of leaving
// the tensor core idle for a quarter (gate|up) to a half (down projection) of every tile.  Plain launches only: no
// split-K, no fused collective, bf16 results through the vectorised epilogue; dense, batched or grouped (segment table,
// expert list or (expert, tile) list).  Tile order: the n_x feature tiles of one token tile are adjacent, so the CTAs
// running at one time share that token tile in L2.
// ---------------------------------------------------------------------------------------------
template <int BN, bool DUAL>
struct PCfg {
    static constexpr int A_BYTES = BM * BK * 2;
    static constexpr int B_BYTES = BN * BK * 2;
    static constexpr int STAGE_BYTES = (DUAL ? 2 : 1) * A_BYTES + B_BYTES;
    static constexpr int STAGING_BYTES = 2 * 16 * BM * 4;          // two [16 tokens][128 features] fp32 transposes
    static constexpr int STAGES_RAW = (210 * 1024 - STAGING_BYTES) / STAGE_BYTES;
    static constexpr int STAGES = STAGES_RAW > 8 ? 8 : STAGES_RAW;
    static constexpr int ACC_COLS = BN * (DUAL ? 2 : 1);
    static constexpr int TMEM_COLS = 2 * ACC_COLS <= 256 ? 256 : 512;
    static constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + STAGING_BYTES + 1024 /*align*/ + 256 /*barriers*/;
    static_assert(2 * ACC_COLS <= 512, "two accumulator sets must fit tensor memory");
    static_assert(ACC_COLS >= 128, "the persistent form is for wide token tiles");
};

struct PTile {
    int n0, batch, row0, rows_valid, row_base;
};

// Work item -> tile; false: nothing to do (an expert without rows, an unused list slot, a token tile past the segment).
template <int BN>
__device__ __forceinline__ bool ptile_decode(const GemmArgs & args, int item, int n_x, int n_y, PTile & t) {
    const int x = item % n_x, rest = item / n_x;
    const int y = rest % n_y, slot = rest / n_y;
    t.n0 = x * BM;
    t.batch = slot;
    t.row0 = y * BN;
    t.rows_valid = args.T;
    t.row_base = 0;
    if (args.seg != nullptr) {
        if (args.expert_list != nullptr) {
            t.batch = args.expert_list[slot];
            if (args.list_tiles && t.batch >= 0) {
                t.row0 = (t.batch >> 16) * BN;
                t.batch &= 0xffff;
            }
        }
        if (t.batch < 0) return false;
        t.row_base = args.seg[t.batch];
        t.rows_valid = args.seg[t.batch + 1] - t.row_base;
    }
    return t.row0 < t.rows_valid;
}

template <int BN, bool DUAL, int FN>
__global__ void __launch_bounds__(NUM_THREADS, 1)
gemm_persistent_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmA2,
                       const __grid_constant__ CUtensorMap tmB, const GemmArgs args, const int n_x, const int n_y, const int n_items) {
    using C = PCfg<BN, DUAL>;
    extern __shared__ uint8_t smem_raw[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    uint8_t * tiles = (uint8_t *) (((uintptr_t) smem_raw + 1023) & ~(uintptr_t) 1023);
    float * staging = (float *) (tiles + C::STAGES * C::STAGE_BYTES);
    uint64_t * bars = (uint64_t *) ((uint8_t *) staging + C::STAGING_BYTES);
    uint64_t * full = bars;
    uint64_t * empty = bars + C::STAGES;
    uint64_t * acc_ready = bars + 2 * C::STAGES;          // [2]
    uint64_t * acc_empty = acc_ready + 2;                 // [2]
    uint32_t * tmem_slot = (uint32_t *) (acc_empty + 2);

    if (threadIdx.x == 0) {
        for (int s = 0; s < C::STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&acc_ready[b], 1); mbar_init(&acc_empty[b], 4); }
        fence_barrier_init();
        prefetch_tmap(&tmA);
        prefetch_tmap(&tmB);
        if (DUAL) prefetch_tmap(&tmA2);
    }
    // This kernel may take every tensor-memory column of its SM (tcgen05.alloc blocks until they are free): it asks only
    // after the grid before it has completed and releases the grid after it only once it holds its columns.
    pdl_wait();
    if (warp == 1) {
        tmem_alloc(tmem_slot, C::TMEM_COLS);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    pdl_launch_dependents();
    const uint32_t tmem = *tmem_slot;
    const int num_kb = (args.K + BK - 1) / BK;

    if (warp == 0) {
        // ================= TMA producer =================
        if (elect_one()) {
            uint32_t it = 0;
            bool ok = true;
            for (int item = blockIdx.x; item < n_items && ok; item += gridDim.x) {
                PTile t;
                if (!ptile_decode<BN>(args, item, n_x, n_y, t)) continue;
                const int b_z = args.seg != nullptr ? 0 : t.batch;
                const int b_row = t.row_base + t.row0;
                for (int kb = 0; kb < num_kb; ++kb, ++it) {
                    const int s = it % C::STAGES;
                    const uint32_t ph = (it / C::STAGES) & 1;
                    if (!mbar_wait(&empty[s], ph ^ 1)) { jib_report(args.status, JIB_ERR_WAIT_TIMEOUT, 11, item); ok = false; break; }
                    uint8_t * st = tiles + s * C::STAGE_BYTES;
                    mbar_expect_tx(&full[s], C::STAGE_BYTES);
                    tma_load_3d(st, &tmA, &full[s], kb * BK, t.n0, t.batch);
                    if (DUAL) tma_load_3d(st + C::A_BYTES, &tmA2, &full[s], kb * BK, t.n0, t.batch);
                    tma_load_3d(st + (DUAL ? 2 : 1) * C::A_BYTES, &tmB, &full[s], kb * BK, b_row, b_z);
                }
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        // ================= MMA issuer =================
        if (elect_one()) {
            constexpr uint32_t idesc = idesc_bf16(BM, BN);
            uint32_t it = 0;
            int j = 0;
            bool ok = true;
            for (int item = blockIdx.x; item < n_items && ok; item += gridDim.x) {
                PTile t;
                if (!ptile_decode<BN>(args, item, n_x, n_y, t)) continue;
                const int buf = j & 1;
                // the epilogue of the tile that used this accumulator set two tiles ago has read it
                if (!mbar_wait(&acc_empty[buf], ((j >> 1) & 1) ^ 1)) { jib_report(args.status, JIB_ERR_WAIT_TIMEOUT, 12, item); ok = false; break; }
                tc_fence_after();
                const uint32_t acc = tmem + buf * C::ACC_COLS;
                for (int kb = 0; kb < num_kb; ++kb, ++it) {
                    const int s = it % C::STAGES;
                    const uint32_t ph = (it / C::STAGES) & 1;
                    if (!mbar_wait(&full[s], ph)) { jib_report(args.status, JIB_ERR_WAIT_TIMEOUT, 13, item); ok = false; break; }
                    tc_fence_after();
                    const uint32_t a_addr = smem_u32(tiles + s * C::STAGE_BYTES);
                    const uint32_t b_addr = a_addr + (DUAL ? 2 : 1) * C::A_BYTES;
#pragma unroll
                    for (int kk = 0; kk < BK / UMMA_K; ++kk) {
                        const uint64_t bd = desc_k_sw128(b_addr + kk * UMMA_K * 2);
                        mma_bf16(acc, desc_k_sw128(a_addr + kk * UMMA_K * 2), bd, idesc, (kb | kk) != 0);
                        if (DUAL) mma_bf16(acc + BN, desc_k_sw128(a_addr + C::A_BYTES + kk * UMMA_K * 2), bd, idesc, (kb | kk) != 0);
                    }
                    mma_commit(&empty[s]);
                }
                mma_commit(&acc_ready[buf]);       // also after a failed wait: the epilogue must not wait for good
                ++j;
            }
        }
        __syncwarp();
    } else {
        // ================= epilogue (warps 2..5) =================
        const int q = warp & 3;
        const int r = q * 32 + lane;
        const int ltid = (int) threadIdx.x - 64;
        int j = 0;
        bool ok = true;
        for (int item = blockIdx.x; item < n_items && ok; item += gridDim.x) {
            PTile t;
            if (!ptile_decode<BN>(args, item, n_x, n_y, t)) continue;
            const int buf = j & 1;
            if (!mbar_wait(&acc_ready[buf], (j >> 1) & 1)) { jib_report(args.status, JIB_ERR_WAIT_TIMEOUT, 14, item); ok = false; }
            {
                // the four warps leave together or not at all: they meet at named barrier 1 inside the tile
                uint32_t all;
                asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbar.red.and.pred q, 1, 128, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
                             : "=r"(all) : "r"((uint32_t) ok) : "memory");
                ok = all != 0;
            }
            if (!ok) break;
            tc_fence_after();
            const uint32_t tbase = tmem + buf * C::ACC_COLS + ((uint32_t) (q * 32) << 16);
            const int ncols = min(BN, t.rows_valid - t.row0);
            const long long obase = (long long) t.batch * args.out_batch_stride;
            const long long rbase = (long long) t.batch * args.res_batch_stride;
            const float bias = FN == 3 && t.n0 + r < args.N ? args.bias[t.n0 + r] : 0.f;
#pragma unroll 1
            for (int c = 0; c < BN; c += 16) {
                if (c >= ncols) break;
                uint32_t gv[16], uv[16];
                float by[FN == 2 ? 16 : 1];
                if (FN == 2) {
#pragma unroll
                    for (int k = 0; k < 16; ++k) by[FN == 2 ? k : 0] = row_factor(args, (long long) t.row_base + t.row0 + c + k, c + k < ncols);
                }
                tmem_ld16(tbase + c, gv);
                if (DUAL) tmem_ld16(tbase + BN + c, uv);
                tmem_ld_wait();
                float * sb = staging + ((c >> 4) & 1) * (16 * BM);
#pragma unroll
                for (int k = 0; k < 16; ++k) {
                    const float g = __uint_as_float(gv[k]);
                    sb[k * BM + r] = DUAL ? gated(g, args.act) * __uint_as_float(uv[k])
                                          : function_of<FN>(g, args, FN == 2 ? by[FN == 2 ? k : 0] : bias);
                }
                asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll 1
                for (int h = 0; h < 2; ++h) {
                    const int tok = (ltid >> 4) + h * 8, fg = (ltid & 15) * 8;
                    const int col = c + tok, nn = t.n0 + fg;
                    if (col >= ncols || nn >= args.N) continue;
                    const long long row = t.row_base + t.row0 + col;
                    if (row >= args.rows_total) { jib_report(args.status, JIB_ERR_BOUNDS, 15, (int) row); continue; }
                    float4 a = *(const float4 *) (sb + tok * BM + fg), b = *(const float4 *) (sb + tok * BM + fg + 4);
                    if (args.residual != nullptr) {
                        const long long ri = rbase + row * args.ldr + nn;
                        if (args.res_f32) {
                            const float4 ra = *(const float4 *) ((const float *) args.residual + ri);
                            const float4 rb = *(const float4 *) ((const float *) args.residual + ri + 4);
                            a.x += ra.x; a.y += ra.y; a.z += ra.z; a.w += ra.w;
                            b.x += rb.x; b.y += rb.y; b.z += rb.z; b.w += rb.w;
                        } else {
                            const uint4 raw = *(const uint4 *) ((const __nv_bfloat16 *) args.residual + ri);
                            const float2 r0 = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.x);
                            const float2 r1 = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.y);
                            const float2 r2 = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.z);
                            const float2 r3 = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.w);
                            a.x += r0.x; a.y += r0.y; a.z += r1.x; a.w += r1.y;
                            b.x += r2.x; b.y += r2.y; b.z += r3.x; b.w += r3.y;
                        }
                    }
                    const uint2 lo = pack_bf16x4(a), hi = pack_bf16x4(b);
                    __nv_bfloat16 * dst = args.row_ptr != nullptr
                                              ? (__nv_bfloat16 *) __ldg((const unsigned long long *) args.row_ptr + row)
                                              : (__nv_bfloat16 *) args.out + obase + row * args.ldo;
                    if (dst != nullptr) *(uint4 *) (dst + nn) = make_uint4(lo.x, lo.y, hi.x, hi.y);
                }
            }
            // this warp's tensor-memory reads of the set are complete: hand it back to the MMA issuer
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[buf]);
            asm volatile("bar.sync 1, 128;" ::: "memory");       // the staging buffers start over with the next tile
            ++j;
        }
    }

    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, C::TMEM_COLS);
}

// ---------------------------------------------------------------------------------------------
// host side
// ---------------------------------------------------------------------------------------------
typedef CUresult (*EncodeTiledFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *,
                                  const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiledFn encode_fn() {
    static EncodeTiledFn fn = nullptr;
    static std::once_flag once;
    std::call_once(once, [] {
        void * p = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &qres) == cudaSuccess &&
            qres == cudaDriverEntryPointSuccess)
            fn = (EncodeTiledFn) p;
    });
    return fn;
}

struct MapKey {
    const void * ptr;
    long long rows, cols, batch, row_stride, batch_stride;
    int box_rows;
    bool operator==(const MapKey & o) const { return memcmp(this, &o, sizeof(MapKey)) == 0; }
};
struct MapKeyHash {
    size_t operator()(const MapKey & k) const {
        const uint64_t * p = (const uint64_t *) &k;
        size_t h = 1469598103934665603ull;
        for (size_t i = 0; i < sizeof(MapKey) / 8; ++i) h = (h ^ p[i]) * 1099511628211ull;
        return h;
    }
};

// bf16 matrix [batch][rows][cols] with element strides; box = {64 cols, box_rows, 1}; 128B swizzle.
int make_map(CUtensorMap * out, const void * ptr, long long rows, long long cols, long long batch, long long row_stride,
             long long batch_stride, int box_rows) {
    static std::mutex mu;
    static std::unordered_map<MapKey, CUtensorMap, MapKeyHash> cache;
    MapKey key;
    memset(&key, 0, sizeof(key));
    key.ptr = ptr; key.rows = rows; key.cols = cols; key.batch = batch; key.row_stride = row_stride;
    key.batch_stride = batch_stride; key.box_rows = box_rows;
    {
        std::lock_guard<std::mutex> g(mu);
        auto it = cache.find(key);
        if (it != cache.end()) { *out = it->second; return 0; }
    }
    EncodeTiledFn fn = encode_fn();
    if (!fn) return JIB_E_DRIVER;
    if (((uintptr_t) ptr & 15) || (row_stride * 2) % 16 || (batch > 1 && (batch_stride * 2) % 16)) return JIB_E_ALIGN;
    cuuint64_t dims[3] = {(cuuint64_t) cols, (cuuint64_t) rows, (cuuint64_t) (batch > 0 ? batch : 1)};
    cuuint64_t strides[2] = {(cuuint64_t) row_stride * 2, (cuuint64_t) (batch > 1 ? batch_stride : rows * row_stride) * 2};
    cuuint32_t box[3] = {(cuuint32_t) BK, (cuuint32_t) box_rows, 1};
    cuuint32_t estr[3] = {1, 1, 1};
    CUresult r = fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void *>(ptr), dims, strides, box, estr,
                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                    CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return JIB_E_TENSORMAP;
    std::lock_guard<std::mutex> g(mu);
    if (cache.size() > 65536) cache.clear();
    cache.emplace(key, *out);
    return 0;
}

// JIB_GEMM_CLUSTER=0 keeps split-K on the global-scratch path (A/B comparison, tests of both paths).
bool jib_no_cluster() {
    static const bool off = [] {
        const char * e = getenv("JIB_GEMM_CLUSTER");
        return e != nullptr && e[0] == '0';
    }();
    return off;
}

// JIB_SPLIT_SMALL=1: split-K also for tiles of 8 k-blocks and fewer (A/B measurements).
bool jib_split_small() {
    static const bool on = [] {
        const char * e = getenv("JIB_SPLIT_SMALL");
        return e != nullptr && e[0] == '1';
    }();
    return on;
}

// JIB_EVICT_FIRST=0: weight loads use the default L2 policy (A/B measurements).
bool jib_no_evict_first() {
    static const bool off = [] {
        const char * e = getenv("JIB_EVICT_FIRST");
        return e != nullptr && e[0] == '0';
    }();
    return off;
}

// Automatic split-K count: fill the machine when there are too few output tiles.  base_ctas: CTAs without a split;
// one wave holds sms CTAs (twice that for the narrow token tiles, which share an SM in pairs).
int auto_splits(long long base_ctas, int num_kb, int bn, int sms) {
    int splits = 1;
    const int slots = sms * (bn <= 32 ? 2 : 1);
    if (2 * base_ctas <= slots) {
        splits = (int) (slots / base_ctas);
        if (splits > num_kb / 4) splits = num_kb / 4;      // at least 4 k-blocks (256 K) per split
        // a split costs ~3 us (partials parked, cluster barrier, remote reads); one CTA streams ~64 KB of weights per
        // microsecond, so tiles of up to 8 k-blocks (128 KB single, 256 KB gate|up) are quicker unsplit
        if (num_kb <= 8 && !jib_split_small()) splits = 1;
        if (splits < 1) splits = 1;
    }
    return splits;
}

template <int BN, bool DUAL, int FN>
int launch_as(const CUtensorMap & a, const CUtensorMap & a2, const CUtensorMap & b, const GemmArgs & args, dim3 grid,
           cudaStream_t stream) {
    using C = Cfg<BN, DUAL>;
    static std::atomic<unsigned char> attr_done[jib::MAX_DEVICES];
    if (!jib::ensure_dyn_smem(gemm_kernel<BN, DUAL, FN>, C::SMEM_BYTES, attr_done)) return JIB_E_LAUNCH;
    const cudaError_t e = jib::launch_pdl_cluster(gemm_kernel<BN, DUAL, FN>, grid, dim3(NUM_THREADS), C::SMEM_BYTES, stream,
                                                  args.cluster_split ? args.splits : 1, a, a2, b, args);
    if (e != cudaSuccess) { (void) cudaGetLastError(); return JIB_E_LAUNCH; }
    return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH;
}

template <int BN, bool DUAL>
int launch(const CUtensorMap & a, const CUtensorMap & a2, const CUtensorMap & b, const GemmArgs & args, dim3 grid, cudaStream_t stream) {
    if (!DUAL && args.bias != nullptr) return launch_as<BN, DUAL, DUAL ? 0 : 3>(a, a2, b, args, grid, stream);
    if (!DUAL && args.unary == JIB_UNARY_GELU) return launch_as<BN, DUAL, DUAL ? 0 : 2>(a, a2, b, args, grid, stream);
    if (!DUAL && args.unary != JIB_UNARY_NONE) return launch_as<BN, DUAL, DUAL ? 0 : 1>(a, a2, b, args, grid, stream);
    return launch_as<BN, DUAL, 0>(a, a2, b, args, grid, stream);
}

template <int BN, bool DUAL, int FN>
int launch_persistent_as(const CUtensorMap & a, const CUtensorMap & a2, const CUtensorMap & b, const GemmArgs & args, int n_x, int n_y,
                      long long n_items, int sms, cudaStream_t stream) {
    using C = PCfg<BN, DUAL>;
    static std::atomic<unsigned char> attr_done[jib::MAX_DEVICES];
    if (!jib::ensure_dyn_smem(gemm_persistent_kernel<BN, DUAL, FN>, C::SMEM_BYTES, attr_done)) return JIB_E_LAUNCH;
    const int grid = (int) (n_items < sms ? n_items : sms);
    const cudaError_t e = jib::launch_pdl(gemm_persistent_kernel<BN, DUAL, FN>, dim3(grid), dim3(NUM_THREADS), C::SMEM_BYTES, stream, a, a2, b, args,
                                          n_x, n_y, (int) n_items);
    if (e != cudaSuccess) { (void) cudaGetLastError(); return JIB_E_LAUNCH; }
    return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH;
}

template <int BN, bool DUAL>
int launch_persistent(const CUtensorMap & a, const CUtensorMap & a2, const CUtensorMap & b, const GemmArgs & args, int n_x, int n_y,
                      long long n_items, int sms, cudaStream_t stream) {
    if (!DUAL && args.bias != nullptr) return launch_persistent_as<BN, DUAL, DUAL ? 0 : 3>(a, a2, b, args, n_x, n_y, n_items, sms, stream);
    if (!DUAL && args.unary == JIB_UNARY_GELU) return launch_persistent_as<BN, DUAL, DUAL ? 0 : 2>(a, a2, b, args, n_x, n_y, n_items, sms, stream);
    if (!DUAL && args.unary != JIB_UNARY_NONE) return launch_persistent_as<BN, DUAL, DUAL ? 0 : 1>(a, a2, b, args, n_x, n_y, n_items, sms, stream);
    return launch_persistent_as<BN, DUAL, 0>(a, a2, b, args, n_x, n_y, n_items, sms, stream);
}

// JIB_GEMM_PERSIST=0: launches with several waves of tiles use the one-tile-per-CTA kernel as well (A/B measurements).
bool jib_no_persist() {
    static const bool off = [] {
        const char * e = getenv("JIB_GEMM_PERSIST");
        return e != nullptr && e[0] == '0';
    }();
    return off;
}

}  // namespace

JIB_TL_DEFINE_SETTER(gemm)

extern "C" JIB_EXPORT int jib_gemm_bf16(const jib_gemm_desc * d, void * stream_) {
    cudaStream_t stream = (cudaStream_t) stream_;
    if (d->T <= 0 || d->N <= 0 || d->K <= 0) return 0;
    const bool dual = d->w2 != nullptr;
    const bool grouped = d->seg != nullptr;
    const int batch = d->batch > 0 ? d->batch : 1;
    const bool src_mode = d->src_token != nullptr;
    if (src_mode && (!grouped || d->src_rows <= 0 || d->src_rows > 256 || d->ar != nullptr)) return JIB_E_ARG;
    const int rows_bound = src_mode ? d->src_rows : grouped ? (d->max_rows > 0 ? d->max_rows : d->T) : d->T;
    int bn = d->bn;
    if (bn == 0) {
        bn = 16;
        while (bn < rows_bound && bn < 256) bn *= 2;
        if (dual && bn > 128) bn = 128;     // keeps three pipeline stages in shared memory
    }
    const int n_tiles = (d->N + BM - 1) / BM;
    const int sms = d->sm_count > 0 ? d->sm_count : 148;
    if (d->bn == 0 && bn == 256 && !grouped && d->ar == nullptr && !d->out_f32 && !jib_no_persist()) {
        // Between one and two waves of 256-token tiles the second wave runs half empty and every CTA pays its prologue and
        // epilogue in the open; the same product as 128-token tiles fills the persistent kernel's two to four rounds evenly
        // with the epilogues hidden (2048 x 2048 x 2048: 25 us -> the persistent form).
        const long long t256 = (long long) n_tiles * ((rows_bound + 255) / 256) * batch;
        if (t256 < 2LL * sms && 4 * t256 >= 3LL * sms) bn = 128;
    }
    const int t_tiles = (rows_bound + bn - 1) / bn;
    const int num_kb = (d->K + BK - 1) / BK;
    // split-K: fill the machine when there are too few output tiles
    int splits = d->splits;
    const long long base_ctas = (long long) n_tiles * t_tiles * (grouped ? (d->active_hint > 0 ? d->active_hint : batch) : batch);
    if (splits <= 0) splits = d->scratch != nullptr ? auto_splits(base_ctas, num_kb, bn, d->sm_count > 0 ? d->sm_count : 148) : 1;
    // Two ways to add the splits up: inside a thread-block cluster through distributed shared memory (at most 8 CTAs,
    // cheap reduction) or through a global scratch with a last-arriver reduction (any count).  Measured per decode GEMM
    // on B200: with few tiles (qkv_a 17-29, q_b 24, shared / dense down 16) the cluster wins by 0.5-2.7 us; with 40
    // tiles x 7 splits (o_proj at TP8) the scratch path is 4.4 us faster.  An explicit split count of up to 8 always
    // takes the cluster (tests exercise both).  Launches with up to 4 splits keep the cluster as well (that is the
    // configuration the single-GPU numbers were measured with).
    const bool cluster_ok = !jib_no_cluster() && (d->splits > 0 ? d->splits <= 8 : (base_ctas <= 32 || splits <= 4));
    if (d->splits <= 0 && cluster_ok && splits > 8) splits = 8;     // a portable cluster holds at most 8 CTAs
    if (splits > num_kb) splits = num_kb;
    int kbps = (num_kb + splits - 1) / splits;
    splits = (num_kb + kbps - 1) / kbps;                        // no empty split
    const bool cluster_split = cluster_ok && splits > 1 && splits <= 8;
    const bool list_tiles = grouped && d->expert_list != nullptr && d->list_tiles != 0 && d->n_slots > 0;
    if (list_tiles && (batch > 0xffff || d->bn == 0)) return JIB_E_ARG;      // the list was built for one token-tile width
    const int n_slots = list_tiles ? d->n_slots
                                   : (grouped && d->expert_list != nullptr && d->n_slots > 0 && d->n_slots < batch) ? d->n_slots : batch;
    const long long tiles_total = (long long) n_tiles * (list_tiles ? 1 : t_tiles) * n_slots;
    if (splits > 1 && !cluster_split) {
        const size_t need = (size_t) tiles_total * splits * (dual ? 2 : 1) * bn * BM * sizeof(float);
        if (d->scratch == nullptr || need > d->scratch_bytes || tiles_total > d->n_counters) {
            if (d->splits > 0) return JIB_E_SCRATCH;            // explicit request that cannot be met
            splits = 1;
            kbps = num_kb;
        }
    }

    CUtensorMap ma, ma2, mb;
    int rc = make_map(&ma, d->w, d->N, d->K, batch, d->w_row_stride, d->w_batch_stride, BM);
    if (rc) return rc;
    if (dual) {
        rc = make_map(&ma2, d->w2, d->N, d->K, batch, d->w_row_stride, d->w_batch_stride, BM);
        if (rc) return rc;
    } else {
        ma2 = ma;
    }
    const long long x_rows = src_mode ? d->src_rows : grouped ? d->x_rows_total : d->T;
    if (src_mode && t_tiles != 1) return JIB_E_ARG;
    rc = make_map(&mb, d->x, x_rows, d->K, grouped ? 1 : batch, d->x_row_stride, d->x_batch_stride, bn);
    if (rc) return rc;

    GemmArgs a;
    a.out = d->out; a.residual = d->residual; a.seg = d->seg; a.scratch = (float *) d->scratch; a.counters = d->counters;
    a.status = d->status; a.ldo = d->ldo; a.out_batch_stride = d->out_batch_stride; a.ldr = d->ldr;
    a.res_batch_stride = d->res_batch_stride; a.T = src_mode ? d->src_rows : d->T; a.N = d->N; a.K = d->K; a.splits = splits; a.kb_per_split = kbps;
    a.out_f32 = d->out_f32; a.res_f32 = d->res_f32;
    a.rows_total = grouped ? d->x_rows_total : d->T;
    a.scratch_elems = (long long) (d->scratch_bytes / sizeof(float));
    a.ar_on = 0; a.ar_site = 0;
    a.cluster_split = cluster_split ? 1 : 0;
    a.row_ptr = (void * const *) d->out_row_ptr;
    a.src_token = d->src_token;
    a.pdl_flags = grouped ? d->pdl_flags : 0;
    a.expert_list = grouped ? d->expert_list : nullptr;
    a.list_tiles = (grouped && d->expert_list != nullptr && d->list_tiles) ? 1 : 0;
    a.w_evict_first = (t_tiles == 1 && !jib_no_evict_first()) ? 1 : 0;      // one token tile: every weight byte is used once
    // 16-byte result stores: bf16 rows whose feature offsets keep 16-byte alignment (row pointers of the expert-parallel return
    // path are row starts of bf16 matrices with d % 8 == 0, hence aligned as well)
    a.vec_store = (!d->out_f32 && d->N % 8 == 0 && d->ldo % 8 == 0 && d->out_batch_stride % 8 == 0 && ((uintptr_t) d->out & 15) == 0 &&
                   (d->residual == nullptr || (((uintptr_t) d->residual & 15) == 0 && d->ldr % 8 == 0 && d->res_batch_stride % 8 == 0)))
                      ? 1 : 0;
    if (d->ar != nullptr && (((const JibArCtx *) d->ar)->d_max % 8 != 0 || d->out_f32)) a.vec_store = 0;
    a.ag_flags = (const unsigned *) d->ag_flags; a.ag_epoch = (const unsigned *) d->ag_epoch;
    a.ag_rows = d->ag_rows; a.ag_world = d->ag_world; a.ar_rs_rows = d->ar_rs_rows;
    a.ag_spin_limit = d->ar != nullptr ? ((const JibArCtx *) d->ar)->spin_limit : 0;
    if (a.ag_flags != nullptr && (a.ag_epoch == nullptr || a.ag_rows <= 0 || a.ag_world <= 0 || grouped || batch != 1)) return JIB_E_ARG;
    if (a.ar_rs_rows < 0) return JIB_E_ARG;
    if (a.row_ptr != nullptr && (dual || d->out_f32 || d->residual != nullptr || d->ar != nullptr)) return JIB_E_ARG;
    a.act = d->act; a.unary = dual ? JIB_UNARY_NONE : d->unary; a.scale = d->scale; a.softcap = d->softcap; a.row_scale = d->row_scale;
    a.bias = nullptr;
    if (d->residual != nullptr && d->ldr == 0 && d->res_f32 && !dual && !grouped && batch == 1 && d->ar == nullptr && a.unary == JIB_UNARY_NONE) {
        a.bias = (const float *) d->residual;
        a.residual = nullptr;
    }
    a.cap2 = d->softcap > 0.f ? 2.f * d->scale / d->softcap : 0.f;
    if (a.unary != JIB_UNARY_NONE && d->ar != nullptr) return JIB_E_ARG;
    memset(&a.ar, 0, sizeof(a.ar));
    if (d->ar != nullptr) {
        const JibArCtx * ar = (const JibArCtx *) d->ar;
        // large batches, or a reduce-scatter: partials to one owner per tile, result delivered from there
        const bool two_shot = d->T > ar->max_rows || d->ar_rs_rows > 0;
        if (dual || grouped || batch != 1 || d->N > ar->d_max || n_tiles * t_tiles > ar->max_tiles || d->ar_site < 0 ||
            d->ar_site >= ar->n_sites)
            return JIB_E_ARG;
        if (d->N % 4 || ar->d_max % 4 || d->ldo % 4 || (d->residual != nullptr && d->ldr % 4)) return JIB_E_ALIGN;
        if (two_shot && (d->T > ar->max_rows2 || ar->recv2[0] == nullptr || (ar->n_sites & 1) || d->out_f32)) return JIB_E_ARG;
        a.ar = *ar; a.ar_on = two_shot ? 2 : 1; a.ar_site = d->ar_site;
    }
    // Several waves of wide tiles and nothing but a plain product: the persistent kernel (epilogue under the next tile's MMAs)
    if (splits == 1 && a.ar_on == 0 && !src_mode && a.ag_flags == nullptr && a.vec_store && bn >= 128 && !(dual && bn > 128) &&
        2 * tiles_total >= 3LL * sms && tiles_total < (1LL << 30) && !jib_no_persist()) {
        const int n_y = list_tiles ? 1 : t_tiles;
        if (bn == 128) {
            return dual ? launch_persistent<128, true>(ma, ma2, mb, a, n_tiles, n_y, tiles_total, sms, stream)
                        : launch_persistent<128, false>(ma, ma2, mb, a, n_tiles, n_y, tiles_total, sms, stream);
        }
        return launch_persistent<256, false>(ma, ma2, mb, a, n_tiles, n_y, tiles_total, sms, stream);
    }
    dim3 grid(n_tiles, list_tiles ? 1 : t_tiles, n_slots * splits);
#define JIB_GEMM_CASE(BN_)                                                                          \
    case BN_:                                                                                     \
        return dual ? launch<BN_, true>(ma, ma2, mb, a, grid, stream) : launch<BN_, false>(ma, ma2, mb, a, grid, stream);
    switch (bn) {
        JIB_GEMM_CASE(16)
        JIB_GEMM_CASE(32)
        JIB_GEMM_CASE(64)
        JIB_GEMM_CASE(128)
        case 256:
            if (dual) return JIB_E_ARG;
            return launch<256, false>(ma, ma2, mb, a, grid, stream);
        default:
            return JIB_E_ARG;
    }
#undef JIB_GEMM_CASE
}

// ---------------------------------------------------------------------------------------------
// Allocation-free variant (declared and documented in jib_noalloc.h).
//
// The split-K scratch is this file-scope device array.  In host code its name is only a handle for the
// runtime, not an address a kernel could use: the device address is obtained once per device with
// cudaGetSymbolAddress (that device current) and passed to the kernel like any other pointer.
// Layout: [partials: JIB_NOALLOC_SCRATCH_BYTES][tile counters: JIB_NOALLOC_MAX_TILES ints][status: 4 ints].
// ---------------------------------------------------------------------------------------------
#include "jib_noalloc.h"

static __device__ __align__(256) unsigned char jib_noalloc_scratch[JIB_NOALLOC_SCRATCH_BYTES + JIB_NOALLOC_MAX_TILES * sizeof(int) + 256];

namespace {

constexpr int NOALLOC_MAX_DEVICES = 64;
unsigned char * g_noalloc_base[NOALLOC_MAX_DEVICES] = {nullptr};
int g_noalloc_sms[NOALLOC_MAX_DEVICES] = {0};
std::mutex g_noalloc_mu;

// Device address of the built-in scratch for the current device and that device's SM count; looked up on first use.
int noalloc_base(unsigned char ** out, int * sms) {
    int dev = -1;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= NOALLOC_MAX_DEVICES) return JIB_E_ARG;
    std::lock_guard<std::mutex> g(g_noalloc_mu);
    if (g_noalloc_base[dev] == nullptr) {
        void * p = nullptr;
        const cudaError_t e = cudaGetSymbolAddress(&p, jib_noalloc_scratch);
        if (e != cudaSuccess || p == nullptr) return JIB_E_DRIVER;
        int n = 0;
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) return JIB_E_DRIVER;
        g_noalloc_sms[dev] = n;
        g_noalloc_base[dev] = (unsigned char *) p;
    }
    *out = g_noalloc_base[dev];
    if (sms != nullptr) *sms = g_noalloc_sms[dev];
    return 0;
}

struct NoallocPlan {
    int bn, n_tiles, num_kb, splits, kbps;
    size_t need;
};

NoallocPlan noalloc_plan(int T, int N, int K, int splits, int sms) {
    NoallocPlan p;
    p.bn = 16;
    while (p.bn < T && p.bn < 256) p.bn *= 2;
    p.n_tiles = (N + BM - 1) / BM;
    p.num_kb = (K + BK - 1) / BK;
    if (splits <= 0) splits = auto_splits(p.n_tiles, p.num_kb, p.bn, sms);      // the rule jib_gemm_bf16 applies
    if (splits > p.num_kb) splits = p.num_kb;
    p.kbps = (p.num_kb + splits - 1) / splits;
    p.splits = (p.num_kb + p.kbps - 1) / p.kbps;
    p.need = p.splits > 1 ? (size_t) p.n_tiles * p.splits * p.bn * BM * sizeof(float) : 0;
    return p;
}

// Tensor map built straight into caller storage (no cache, no host allocation).
int encode_plain(CUtensorMap * out, const void * ptr, long long rows, long long cols, int box_rows) {
    EncodeTiledFn fn = encode_fn();
    if (!fn) return JIB_E_DRIVER;
    if (((uintptr_t) ptr & 15) || (cols * 2) % 16) return JIB_E_ALIGN;
    cuuint64_t dims[3] = {(cuuint64_t) cols, (cuuint64_t) rows, 1};
    cuuint64_t strides[2] = {(cuuint64_t) cols * 2, (cuuint64_t) rows * cols * 2};
    cuuint32_t box[3] = {(cuuint32_t) BK, (cuuint32_t) box_rows, 1};
    cuuint32_t estr[3] = {1, 1, 1};
    const CUresult r = fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void *>(ptr), dims, strides, box, estr,
                          CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                          CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : JIB_E_TENSORMAP;
}

}  // namespace

extern "C" JIB_EXPORT size_t jib_gemm_bf16_noalloc_need(int T, int N, int K, int splits) {
    if (T <= 0 || N <= 0 || K <= 0) return 0;
    int sms = 148;                           // splits == 0 depends on the SM count of the current device
    if (splits <= 0) {
        unsigned char * base = nullptr;
        if (noalloc_base(&base, &sms) != 0) sms = 148;
    }
    return noalloc_plan(T, N, K, splits, sms).need;
}

// Copies the four status words of the most recent jib_gemm_bf16_noalloc call on the current device into out (host memory,
// ideally pinned), in stream order behind that call; allocates nothing.  out[0] != 0 after the stream has been
// synchronised means the kernel recorded a fault (1 = a bounded wait ran out, 2 = an index out of range; out[1] = site).
extern "C" JIB_EXPORT int jib_gemm_bf16_noalloc_status(int * out, void * stream_) {
    if (out == nullptr) return JIB_E_ARG;
    unsigned char * base = nullptr;
    const int rc = noalloc_base(&base, nullptr);
    if (rc) return rc;
    const int * status = (const int *) (base + JIB_NOALLOC_SCRATCH_BYTES) + JIB_NOALLOC_MAX_TILES;
    return cudaMemcpyAsync(out, status, 4 * sizeof(int), cudaMemcpyDeviceToHost, (cudaStream_t) stream_) == cudaSuccess ? 0 : JIB_E_LAUNCH;
}

extern "C" JIB_EXPORT int jib_gemm_bf16_noalloc(const void * x, const void * w, void * out, int T, int N, int K, int splits,
                                                void * stream_) {
    cudaStream_t stream = (cudaStream_t) stream_;
    if (T <= 0 || N <= 0 || K <= 0) return 0;
    if (T > 256 || x == nullptr || w == nullptr || out == nullptr) return JIB_E_ARG;
    unsigned char * base = nullptr;
    int sms = 148;
    int rc = noalloc_base(&base, &sms);      // first call on this device: symbol lookup (keep it outside stream capture)
    if (rc) return rc;
    const NoallocPlan p = noalloc_plan(T, N, K, splits, sms);
    if (p.need > JIB_NOALLOC_SCRATCH_BYTES || p.n_tiles > JIB_NOALLOC_MAX_TILES) return JIB_E_NOALLOC_TOO_LARGE;
    int * counters = (int *) (base + JIB_NOALLOC_SCRATCH_BYTES);
    int * status = counters + JIB_NOALLOC_MAX_TILES;
    // the array keeps whatever the previous call left: counters (and the status words) must start at zero
    if (cudaMemsetAsync(counters, 0, (size_t) p.n_tiles * sizeof(int), stream) != cudaSuccess) return JIB_E_LAUNCH;
    if (cudaMemsetAsync(status, 0, 4 * sizeof(int), stream) != cudaSuccess) return JIB_E_LAUNCH;

    CUtensorMap ma, mb;
    rc = encode_plain(&ma, w, N, K, BM);
    if (rc) return rc;
    rc = encode_plain(&mb, x, T, K, p.bn);
    if (rc) return rc;
    GemmArgs a;
    a.out = out; a.residual = nullptr; a.seg = nullptr; a.scratch = (float *) base; a.counters = counters; a.status = status;
    a.ldo = N; a.out_batch_stride = 0; a.ldr = 0; a.res_batch_stride = 0; a.T = T; a.N = N; a.K = K; a.splits = p.splits;
    a.kb_per_split = p.kbps; a.out_f32 = 0; a.res_f32 = 0; a.rows_total = T;
    a.scratch_elems = (long long) (JIB_NOALLOC_SCRATCH_BYTES / sizeof(float));
    a.ar_on = 0; a.ar_site = 0;
    a.cluster_split = 0;
    a.row_ptr = nullptr;
    a.src_token = nullptr;
    a.vec_store = 0;
    a.w_evict_first = 0;
    a.pdl_flags = 0;
    a.expert_list = nullptr;
    a.list_tiles = 0;
    a.ag_flags = nullptr; a.ag_epoch = nullptr; a.ag_rows = 0; a.ag_world = 0; a.ar_rs_rows = 0; a.ag_spin_limit = 0;
    a.act = JIB_ACT_SILU; a.unary = JIB_UNARY_NONE; a.scale = 1.f; a.softcap = a.cap2 = 0.f; a.row_scale = a.bias = nullptr;
    memset(&a.ar, 0, sizeof(a.ar));
    dim3 grid(p.n_tiles, 1, p.splits);
    switch (p.bn) {
        case 16: return launch<16, false>(ma, ma, mb, a, grid, stream);
        case 32: return launch<32, false>(ma, ma, mb, a, grid, stream);
        case 64: return launch<64, false>(ma, ma, mb, a, grid, stream);
        case 128: return launch<128, false>(ma, ma, mb, a, grid, stream);
        case 256: return launch<256, false>(ma, ma, mb, a, grid, stream);
        default: return JIB_E_ARG;
    }
}
