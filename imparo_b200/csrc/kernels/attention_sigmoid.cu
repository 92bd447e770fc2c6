// Attention whose weights are sigmoids instead of a softmax: a visible key weighs
//
//     w = sigmoid(scale * q.k + bias_h)          (bias_h: a number per query head; weights are not normalised over the keys)
//
// over the paged cache in bfloat16, for masks that keep all earlier positions, a sliding window, or the position's own stretch
// of `chunk` positions (first_key, common.cuh).  Without a maximum and a denominator a row's output is a plain sum over its
// keys, so it stays in tensor memory across the steps and is never rescaled, and partial sums over key ranges simply add.
//
//  (1) attn_sigmoid_prefill: prompt portions on the 5th-generation tensor cores.  Key size and value size each a multiple of
//      16 up to 128 (they need not be equal), up to 128 query heads per kv head, pages of 16, 32, 64 or 128 positions.  A CTA
//      owns up to 128 query rows, (128 / G) consecutive tokens of ONE request times the G query heads of a kv head:
//        warp 0      TMA: the step's 128 keys and values page by page (128-byte swizzle) into a ring of two stages
//        warp 1      tcgen05.mma: S = Q K^T into tensor memory, issued for the next step as soon as the scores have been read;
//                    O += P V accumulated in tensor memory when the step's weights are written
//        warps 2-9   two threads per row (half of the step's keys each): scores to registers, mask, weights as bfloat16
//                    into shared memory in the MMA's swizzled layout; at the end the row's output
//  (2) attn_sigmoid_split: single query tokens.  A CTA takes one range of keys (counted from the query's first key), one kv
//      head and one token, scores and sums with mma.sync m16n8k16 for the group's heads at once, and leaves its partial sum;
//      the partials carry (0, 1 / ranges) where a softmax's carry (max, sum), so that the ordered combine of the softmax
//      kernels (attention_split.cu, or inside the output product) adds them up.
//
// The weights are computed in 32-bit: 1 / (1 + 2^t), t = -(scale q.k + bias) log2 e limited to 60 (the weight is below 1e-18
// there), two reciprocals from one (1/a = b/(ab), 1/b = a/(ab)): the special-function units are what limits a step.
//
// Every wait on an mbarrier is bounded: when it runs out the kernel records IMPARO_ST_WAIT_LIMIT in the status word, stops
// waiting, frees its tensor memory and returns.
#include "tcgen05.cuh"

namespace imparo {
namespace sg {

using namespace tc;

constexpr int ROWS = 128, KEYS = 128, THREADS = 320, STAGES = 2;
constexpr uint32_t REGION = 128 * 128;      // a [128 rows][128 bytes] block of a tile: 16 KB
constexpr uint32_t ALIGN_SLACK = 768;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t addr, uint32_t lbo_bytes) {
    // values as B operand: [key][dim] with the dims contiguous, 128-byte swizzle: groups of 8 keys 1024 bytes apart, 64-dim
    // blocks lbo bytes apart
    uint64_t d = 0;
    d |= (uint64_t)((addr & 0x3FFFF) >> 4);
    d |= (uint64_t)((lbo_bytes >> 4) & 0x3FFF) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
__device__ __forceinline__ uint32_t instr_desc_ab(int m, int n, bool b_mn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn ? (1u << 16) : 0u) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
// the weights of two scores: s * nsl2 + nb2 = -(scale s + bias) log2 e
__device__ __forceinline__ void weights2(float s0, float s1, float nsl2, float nb2, float& p0, float& p1) {
    const float a = 1.0f + ex2(fminf(fmaf(s0, nsl2, nb2), 60.f)), b = 1.0f + ex2(fminf(fmaf(s1, nsl2, nb2), 60.f));
    const float r = rcp(a * b);
    p0 = r * b;
    p1 = r * a;
}
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}

struct Args {
    const __nv_bfloat16* q;
    __nv_bfloat16* out;
    const int* item_row_start;
    const int* item_start_pos;
    const int* table;
    const float* bias;
    int* status;
    int n_items, max_blocks, page_size, n_pages, window, chunk, nh, nkv, hd, vd;
    float scale;
};

// NBK, NBV: 64-dim blocks of a key head and of a value head
template <int NBK, int NBV>
__global__ void __launch_bounds__(THREADS, NBK + NBV == 2 ? 2 : 1)
prefill_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, const Args a) {
    constexpr uint32_t Q_BYTES = NBK * REGION, P_BYTES = 2 * REGION, K_BYTES = NBK * REGION, V_BYTES = NBV * REGION;
    constexpr uint32_t STAGE_BYTES = K_BYTES + V_BYTES, TMEM_COLS = 256;      // scores: columns 0..127, output: 128..
    extern __shared__ __align__(1024) uint8_t sg_smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>(((uintptr_t)sg_smem_raw + 1023) & ~(uintptr_t)1023);
    if ((uint32_t)(smem - sg_smem_raw) > ALIGN_SLACK) {      // the launch's shared memory does not cover the aligned tiles
        if (threadIdx.x == 0) report(a.status, IMPARO_ST_WAIT_LIMIT, 109, (int)(smem - sg_smem_raw), 0);
        return;
    }
    uint8_t* q_s = smem;
    uint8_t* p_s = q_s + Q_BYTES;
    uint8_t* kv_s = p_s + P_BYTES;                           // [stage][K | V]
    uint64_t* kv_full = reinterpret_cast<uint64_t*>(kv_s + STAGES * STAGE_BYTES);      // [STAGES]
    uint64_t* kv_empty = kv_full + STAGES;                   // [STAGES]
    uint64_t* q_ready = kv_empty + STAGES;
    uint64_t* s_ready = q_ready + 1;                         // a step's scores are complete
    uint64_t* s_free = q_ready + 2;                          // ... and have been read
    uint64_t* p_ready = q_ready + 3;                         // the step's weights are written
    uint64_t* o_done = q_ready + 4;                          // their P V is accumulated
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_ready + 5);

    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int G = a.nh / a.nkv, TQ = ROWS / G;
    const int kvh = blockIdx.x;
    // tiles are numbered request by request; they run backwards along the slow grid index (the ones with the most keys first)
    int item = 0, tile = (int)gridDim.y - 1 - (int)blockIdx.y, n_item = 0, row0 = 0;
    for (; item < a.n_items; ++item) {
        row0 = a.item_row_start[item];
        n_item = a.item_row_start[item + 1] - row0;
        const int tiles = (n_item + TQ - 1) / TQ;
        if (tile < tiles) break;
        tile -= tiles;
    }
    if (item >= a.n_items) {                                 // the grid is an upper bound (uniform per CTA)
        if (threadIdx.x == 0) pdl_wait();
        return;
    }
    const int tok0 = tile * TQ, n_tok = min(TQ, n_item - tok0), n_rows = n_tok * G;
    const int pos0 = a.item_start_pos[item] + tok0, pos_last = pos0 + n_tok - 1;
    const int* tab = a.table + (size_t)item * a.max_blocks;
    const int lo_min = first_key(pos0, a.window, a.chunk);
    const int kb_first = lo_min / KEYS, n_steps = pos_last / KEYS - kb_first + 1;

    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) { mbar_init(&kv_full[s], 1); mbar_init(&kv_empty[s], 1); }
        mbar_init(q_ready, 256);
        mbar_init(s_ready, 1);
        mbar_init(s_free, 256);
        mbar_init(p_ready, 256);
        mbar_init(o_done, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        // lane 0 waits for the stage and sets the byte count, lane p looks up page p of the step and issues its copies
        pdl_wait();                                          // this step's keys were written by the kernel before
        const int pages_per_step = KEYS / a.page_size;
        const int first_blk = lo_min / a.page_size, last_blk = pos_last / a.page_size;
        int issued = 0;
        for (int i = 0; i < n_steps; ++i) {
            const int s = i % STAGES;
            int ok = 1;
            if (lane == 0) {
                if (i >= STAGES && !mbar_wait(&kv_empty[s], ((i / STAGES) - 1) & 1)) {
                    report(a.status, IMPARO_ST_WAIT_LIMIT, 101, i, s);
                    ok = 0;
                } else {
                    mbar_expect_tx(&kv_full[s], STAGE_BYTES);
                }
            }
            ok = __shfl_sync(0xffffffffu, ok, 0);            // (also orders the byte count before the copies)
            if (!ok) break;
            uint8_t* kdst = kv_s + s * STAGE_BYTES;
            uint8_t* vdst = kdst + K_BYTES;
            const int blk0 = (kb_first + i) * pages_per_step;
            for (int pg = lane; pg < pages_per_step; pg += 32) {
                // a block before every row's first key (its page may be gone) or past the last position holds nothing
                // this tile may use: a mapped page stands in for it (its keys are masked, its values finite)
                const int blk = min(max(blk0 + pg, first_blk), last_blk);
                int page = blk < a.max_blocks ? tab[blk] : -1;
                if (page < 0 || page >= a.n_pages) {
                    report(a.status, IMPARO_ST_PAGE_RANGE, 102, item, page);
                    page = 0;
                }
                const int y = page * a.page_size;
                const uint32_t off = (uint32_t)pg * a.page_size * 128;
#pragma unroll
                for (int nb = 0; nb < NBK; ++nb) tma_load_2d(kdst + nb * REGION + off, &map_k, &kv_full[s], kvh * a.hd + nb * 64, y);
#pragma unroll
                for (int nb = 0; nb < NBV; ++nb) tma_load_2d(vdst + nb * REGION + off, &map_v, &kv_full[s], kvh * a.vd + nb * 64, y);
            }
            issued = i + 1;
        }
        // nobody leaves while copies are in flight (they have landed already unless a wait ran out somewhere)
        if (lane == 0)
            for (int i = max(0, issued - STAGES); i < issued; ++i) mbar_wait(&kv_full[i % STAGES], (i / STAGES) & 1);
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = instr_desc_ab(ROWS, KEYS, false);
            const uint32_t idesc_o = instr_desc_ab(ROWS, NBV * 64, true);      // whole 64-dim blocks (columns past vd are not read)
            const uint32_t t_s = tmem_base, t_o = tmem_base + 128;
            const uint32_t qb = smem_u32(q_s), pb = smem_u32(p_s);
            const int ksteps = a.hd / UMMA_K;
            auto wait_for = [&](uint64_t* bar, uint32_t parity, int code, int i) -> bool {
                if (mbar_wait(bar, parity)) { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); return true; }
                report(a.status, IMPARO_ST_WAIT_LIMIT, code, i, 0);
                return false;
            };
            auto issue_s = [&](int i) {                       // S = Q K_i^T
                const uint32_t kb = smem_u32(kv_s + (i % STAGES) * STAGE_BYTES);
                for (int k = 0; k < ksteps; ++k)
                    umma(t_s, smem_desc(qb + (k >> 2) * REGION + (k & 3) * 32), smem_desc(kb + (k >> 2) * REGION + (k & 3) * 32), idesc_s,
                         k > 0 ? 1u : 0u);
                umma_commit(s_ready);
            };
            auto issue_pv = [&](int i) {                      // O += P_i V_i
                const uint32_t vb = smem_u32(kv_s + (i % STAGES) * STAGE_BYTES + K_BYTES);
#pragma unroll
                for (int kk = 0; kk < KEYS / UMMA_K; ++kk)
                    umma(t_o, smem_desc(pb + (kk >> 2) * REGION + (kk & 3) * 32), smem_desc_mn(vb + kk * (UMMA_K * 128), REGION), idesc_o,
                         (i > 0 || kk > 0) ? 1u : 0u);
                umma_commit(&kv_empty[i % STAGES]);           // keys (scored earlier) and values of the stage are read
                umma_commit(o_done);
            };
            bool ok = wait_for(q_ready, 0, 103, 0) && wait_for(&kv_full[0], 0, 104, 0);
            int s_issued = 0, pv_issued = 0;
            if (ok) { issue_s(0); s_issued = 1; }
            for (int i = 0; i < n_steps && ok; ++i) {
                if (i + 1 < n_steps) {
                    ok = wait_for(s_free, i & 1, 105, i) && wait_for(&kv_full[(i + 1) % STAGES], ((i + 1) / STAGES) & 1, 104, i + 1);
                    if (!ok) break;
                    issue_s(i + 1);
                    s_issued = i + 2;
                }
                ok = wait_for(p_ready, i & 1, 106, i);
                if (ok) { issue_pv(i); pv_issued = i + 1; }
            }
            // ... or products that still write tensor memory
            if (s_issued) mbar_wait(s_ready, (s_issued - 1) & 1);
            if (pv_issued) mbar_wait(o_done, (pv_issued - 1) & 1);
        }
    } else {
        const int half = (warp - 2) >> 2;                     // keys 0-63 or 64-127 of a step
        const int r = (warp & 3) * 32 + lane;                 // the row: a tensor-memory lane
        const bool valid = r < n_rows;
        const int tok = r / G, head = kvh * G + r % G;
        const int pos_r = pos0 + tok;
        const int lo_r = first_key(pos_r, a.window, a.chunk), lo_last = first_key(pos_last, a.window, a.chunk);
        const uint32_t t_lane = tmem_base + ((uint32_t)((warp & 3) * 32) << 16);
        const uint32_t t_s = t_lane + half * 64, t_o = t_lane + 128;
        const size_t row = (size_t)(row0 + tok0 + (valid ? tok : 0)) * a.nh + head;
        pdl_wait();
        {
            // this thread's half of the row's queries -> shared memory, 16-byte pieces swizzled as the MMA reads them
            const uint4* src = reinterpret_cast<const uint4*>(a.q + row * a.hd);
            for (int c = half; c < a.hd / 8; c += 2) {
                const uint4 v = valid ? src[c] : make_uint4(0u, 0u, 0u, 0u);
                *reinterpret_cast<uint4*>(q_s + (c >> 3) * REGION + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v;
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            mbar_arrive(q_ready);
        }
        const float nsl2 = -a.scale * LOG2E, nb2 = -a.bias[valid ? head : 0] * LOG2E;
        uint8_t* prow = p_s + half * REGION + r * 128;        // keys 0-63 and 64-127 are the two blocks of P
        bool ok = true;
        for (int i = 0; i < n_steps; ++i) {
            // (a warp stays whole: what follows are the whole warp's instructions.  One warp giving up leaves the others waiting for
            // its arrivals, and all of their waits are bounded)
            ok = __all_sync(0xffffffffu, mbar_wait(s_ready, i & 1));
            if (!ok) { report(a.status, IMPARO_ST_WAIT_LIMIT, 107, i, r); break; }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            float v[4][16];
            tmem_ld_chunks<4>(t_s, v);
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(s_free);                              // the score columns may take the next step's product
            const int key0 = (kb_first + i) * KEYS + half * 64;
            const int j_hi = valid ? min(63, pos_r - key0) : -1, j_lo = max(0, lo_r - key0);      // the keys this row sees
            const bool whole = (kb_first + i) * KEYS + KEYS - 1 <= pos0 && (kb_first + i) * KEYS >= lo_last && valid;
            uint32_t w[32];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
#pragma unroll
                for (int e = 0; e < 16; e += 2) {
                    float p0, p1;
                    weights2(v[u][e], v[u][e + 1], nsl2, nb2, p0, p1);
                    w[u * 8 + (e >> 1)] = pack2(p0, p1);
                }
            }
            if (!whole) {
#pragma unroll
                for (int k = 0; k < 32; ++k) {
                    const uint32_t m = ((2 * k >= j_lo && 2 * k <= j_hi) ? 0x0000ffffu : 0u) | ((2 * k + 1 >= j_lo && 2 * k + 1 <= j_hi) ? 0xffff0000u : 0u);
                    w[k] &= m;
                }
            }
            // the step before has read its weights out of the buffer
            ok = __all_sync(0xffffffffu, i == 0 || mbar_wait(o_done, (i - 1) & 1));
            if (!ok) { report(a.status, IMPARO_ST_WAIT_LIMIT, 108, i, r); break; }
#pragma unroll
            for (int c = 0; c < 8; ++c)
                *reinterpret_cast<uint4*>(prow + ((c ^ (r & 7)) << 4)) = make_uint4(w[4 * c], w[4 * c + 1], w[4 * c + 2], w[4 * c + 3]);
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            mbar_arrive(p_ready);
        }
        if (ok) {
            ok = __all_sync(0xffffffffu, mbar_wait(o_done, (n_steps - 1) & 1));
            if (!ok) report(a.status, IMPARO_ST_WAIT_LIMIT, 108, n_steps, r);
        }
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            for (int c = half; c < a.vd / 16; c += 2) {        // 16 columns at a time, the row's two threads in turn
                float o[16];
                tmem_ld16(t_o + c * 16, o);
                if (valid) {
                    uint4* dst = reinterpret_cast<uint4*>(a.out + row * a.vd + c * 16);
                    dst[0] = make_uint4(pack2(o[0], o[1]), pack2(o[2], o[3]), pack2(o[4], o[5]), pack2(o[6], o[7]));
                    dst[1] = make_uint4(pack2(o[8], o[9]), pack2(o[10], o[11]), pack2(o[12], o[13]), pack2(o[14], o[15]));
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(TMEM_COLS) : "memory");
    }
}

template <int NBK, int NBV>
static int launch_prefill(const CUtensorMap& mk, const CUtensorMap& mv, const Args& a, dim3 grid, cudaStream_t stream) {
    constexpr size_t smem = ALIGN_SLACK + (size_t)(NBK + 2 + STAGES * (NBK + NBV)) * REGION + 128;
    auto kern = prefill_kernel<NBK, NBV>;
    static bool configured = false;
    cudaError_t e;
    if (!configured) {
        e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    e = launch(kern, grid, dim3(THREADS), smem, stream, mk, mv, a);
    return e == cudaSuccess ? 0 : (int)e;
}

// ---- (2) single query tokens ------------------------------------------------------------------------------------
constexpr int DT = 128, DKEYS = 64;         // threads and keys per step: four warps of 16 keys each

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;                 // 0: the 16 bytes are zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// byte offset of 16-byte piece c of row r in a tile with rows of W elements, XOR-swizzled so that the eight rows an ldmatrix
// reads fall into distinct banks
template <int W> __device__ __forceinline__ uint32_t tile_off(int r, int c) { return (uint32_t)r * (W * 2) + (uint32_t)((c ^ (r & 7)) << 4); }

// KW, VW: the key and value size rounded up to 64 or 128 (the tiles' row width); hd and vd are multiples of 16.
template <int KW, int VW>
__global__ void __launch_bounds__(DT, 3)
split_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache,
             const int* __restrict__ positions, const int* __restrict__ item_of_token, const int* __restrict__ table, int max_blocks,
             int page_size, int n_pages, int window, int chunk, float scale, const float* __restrict__ bias,
             float* __restrict__ part_acc, float* __restrict__ part_ml, int nh, int nkv, int hd, int vd, int range, int n_splits,
             int fresh, int* status) {
    constexpr uint32_t K_BYTES = DKEYS * KW * 2, V_BYTES = DKEYS * VW * 2;
    constexpr int NT = VW / 8, KT = KW / 16;
    extern __shared__ __align__(128) uint8_t sgd_smem[];      // [2][K | V], afterwards the four warps' sums
    pdl_trigger();
    const int split = blockIdx.x, kvh = blockIdx.y, t = blockIdx.z;
    const int G = nh / nkv;
    const int page_shift = (page_size & (page_size - 1)) == 0 ? 31 - __clz(page_size) : -1;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2, tg = lane & 3;
    const int pos = positions[t];
    const int lo = first_key(pos, window, chunk);
    const int begin = lo + split * range, end = min(pos + 1, begin + range);      // ranges are counted from the first key
    const int h0 = kvh * G;
    const size_t part_base = ((size_t)t * nh + h0) * n_splits + split;             // + head of the group * n_splits
    const int* tab = table + (size_t)item_of_token[t] * max_blocks;
    const size_t kw = (size_t)nkv * hd, vw = (size_t)nkv * vd;
    const int n_steps = begin < end ? (end - begin + DKEYS - 1) / DKEYS : 0;
    // two threads per key of a step (alternate 16-byte pieces); a warp fetches the very keys it scores
    auto load_kv = [&](int step, int buf) {
        const int r = tid >> 1, c0 = tid & 1;
        const int j = begin + step * DKEYS + r;
        bool valid = j < end;
        size_t rowi = 0;
        if (valid) {
            const int blk = page_shift >= 0 ? j >> page_shift : j / page_size;
            const int within = page_shift >= 0 ? j & (page_size - 1) : j % page_size;
            const int page = blk < max_blocks ? tab[blk] : -1;
            if (page < 0 || page >= n_pages) {
                if (c0 == 0) report(status, IMPARO_ST_PAGE_RANGE, 110, t, page);
                valid = false;
            } else {
                rowi = (size_t)page * page_size + within;
            }
        }
        uint8_t* const kd = sgd_smem + buf * (K_BYTES + V_BYTES);
        uint8_t* const vd_s = kd + K_BYTES;
        const __nv_bfloat16* ksrc = k_cache + rowi * kw + (size_t)kvh * hd;
        const __nv_bfloat16* vsrc = v_cache + rowi * vw + (size_t)kvh * vd;
#pragma unroll
        for (int c = c0; c < KW / 8; c += 2) {
            const bool in = valid && c * 8 < hd;
            cp_async16(kd + tile_off<KW>(r, c), in ? ksrc + c * 8 : k_cache, in);
        }
#pragma unroll
        for (int c = c0; c < VW / 8; c += 2) {
            const bool in = valid && c * 8 < vd;
            cp_async16(vd_s + tile_off<VW>(r, c), in ? vsrc + c * 8 : v_cache, in);
        }
        cp_commit();
    };
    // rows below pos + 1 - fresh were written by earlier steps: their tiles are requested before the wait
    const int old_end = fresh > 0 ? pos + 1 - fresh : -1;
    int requested = 0;                                        // steps asked for so far
    for (int u = 0; u < 2 && u < n_steps; ++u) {
        if (min(end, begin + (u + 1) * DKEYS) <= old_end) { load_kv(u, u); requested = u + 1; } else break;
    }
    pdl_wait();
    if (n_steps == 0) {
        if (tid < G) {
            part_ml[(part_base + (size_t)tid * n_splits) * 2] = -INFINITY;
            part_ml[(part_base + (size_t)tid * n_splits) * 2 + 1] = 0.f;
        }
        return;
    }
    // the queries in the MMA's A layout: row g of the 16-row tile is head h0 + g (rows from G up are padding)
    uint32_t qf[KT][4];
    {
        const __nv_bfloat16* qrow = q + ((size_t)t * nh + h0 + (g < G ? g : 0)) * hd + 2 * tg;
#pragma unroll
        for (int kt = 0; kt < KT; ++kt) {
            const bool in = g < G && kt * 16 < hd;
            qf[kt][0] = in ? *reinterpret_cast<const uint32_t*>(qrow + kt * 16) : 0u;
            qf[kt][2] = in ? *reinterpret_cast<const uint32_t*>(qrow + kt * 16 + 8) : 0u;
            qf[kt][1] = qf[kt][3] = 0u;
        }
    }
    if (requested == 0) { load_kv(0, 0); requested = 1; }
    const float nsl2 = -scale * LOG2E, nb2 = -(g < G ? bias[h0 + g] : 0.f) * LOG2E;
    float o[NT][2];                                           // rows 0..7 only (G <= 8)
#pragma unroll
    for (int n = 0; n < NT; ++n) { o[n][0] = o[n][1] = 0.f; }
    const int mi = lane >> 3, rin = lane & 7;
    for (int step = 0; step < n_steps; ++step) {
        const int buf = step & 1;
        if (step + 1 < n_steps && requested < step + 2) { load_kv(step + 1, buf ^ 1); requested = step + 2; }
        if (step + 1 < n_steps) cp_wait<1>(); else cp_wait<0>();
        __syncwarp();                                         // the warp's own 16 keys have landed
        const uint8_t* const kt_s = sgd_smem + buf * (K_BYTES + V_BYTES);
        const uint8_t* const vt_s = kt_s + K_BYTES;
        float s[2][4];
        s[0][0] = s[0][1] = s[0][2] = s[0][3] = s[1][0] = s[1][1] = s[1][2] = s[1][3] = 0.f;
        {
            const int key = warp * 16 + (mi >> 1) * 8 + rin;
#pragma unroll
            for (int kt = 0; kt < KT; ++kt) {
                if (kt * 16 < hd) {
                    uint32_t b[4];
                    ldmatrix4(b, smem_u32(kt_s + tile_off<KW>(key, kt * 2 + (mi & 1))));
                    mma16816(s[0], qf[kt], b[0], b[1]);
                    mma16816(s[1], qf[kt], b[2], b[3]);
                }
            }
        }
        const int key0 = begin + step * DKEYS + warp * 16 + 2 * tg;
        float p[2][2];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            weights2(s[n][0], s[n][1], nsl2, nb2, p[n][0], p[n][1]);
#pragma unroll
            for (int e = 0; e < 2; ++e) if (key0 + n * 8 + e >= end) p[n][e] = 0.f;
        }
        {
            const uint32_t a[4] = {pack2(p[0][0], p[0][1]), 0u, pack2(p[1][0], p[1][1]), 0u};      // rows 8..15 are padding
            const int key = warp * 16 + (mi & 1) * 8 + rin;
#pragma unroll
            for (int np = 0; np < NT / 2; ++np) {
                if (np * 16 < vd) {
                    uint32_t b[4];
                    ldmatrix4_trans(b, smem_u32(vt_s + tile_off<VW>(key, np * 2 + (mi >> 1))));
                    float c0[4] = {o[2 * np][0], o[2 * np][1], 0.f, 0.f};
                    float c1[4] = {o[2 * np + 1][0], o[2 * np + 1][1], 0.f, 0.f};
                    mma16816(c0, a, b[0], b[1]);
                    mma16816(c1, a, b[2], b[3]);
                    o[2 * np][0] = c0[0]; o[2 * np][1] = c0[1];
                    o[2 * np + 1][0] = c1[0]; o[2 * np + 1][1] = c1[1];
                }
            }
        }
        __syncwarp();                                         // the warp refills this buffer two steps on
    }
    __syncthreads();                                          // the tiles' bytes become the sums' scratch
    float* acc = reinterpret_cast<float*>(sgd_smem);          // [4 warps][8 heads][VW]
#pragma unroll
    for (int n = 0; n < NT; ++n)
        *reinterpret_cast<float2*>(acc + ((size_t)warp * 8 + g) * VW + n * 8 + 2 * tg) = make_float2(o[n][0], o[n][1]);
    __syncthreads();
    const int live = (pos - lo) / range + 1;                  // ranges of this token that hold keys
    for (int idx = tid; idx < G * vd; idx += DT) {
        const int gg = idx / vd, d = idx - gg * vd;
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) sum += acc[((size_t)w * 8 + gg) * VW + d];
        part_acc[(part_base + (size_t)gg * n_splits) * vd + d] = sum;
        if (d == 0) {
            part_ml[(part_base + (size_t)gg * n_splits) * 2] = 0.f;
            part_ml[(part_base + (size_t)gg * n_splits) * 2 + 1] = 1.0f / (float)live;
        }
    }
}

}  // namespace sg
}  // namespace imparo

using namespace imparo;

// bfloat16; hd and vd multiples of 16 up to 128, at most 128 query heads per kv head, pages of 16, 32, 64 or 128 positions; else
// -8 (the caller uses another kernel).  bias float32 [nh].  The caches are [n_pages * page_size rows, nkv * hd | nkv * vd].
extern "C" int imparo_attention_sigmoid_prefill(const void* q, const void* k_cache, const void* v_cache, const int* item_row_start,
                                                const int* item_start_pos, int n_items, const int* table, int max_blocks, int page_size,
                                                int n_pages, int window, int chunk, float scale, const float* bias, void* out, int n_tok,
                                                int nh, int nkv, int hd, int vd, int* status, cudaStream_t stream) {
    if (n_tok <= 0) return 0;
    if (nkv <= 0 || nh % nkv != 0) return -5;
    const int G = nh / nkv;
    if (G > sg::ROWS || hd < 16 || hd > 128 || hd % 16 || vd < 16 || vd > 128 || vd % 16) return -8;
    if (page_size != 16 && page_size != 32 && page_size != 64 && page_size != 128) return -8;
    if (((uintptr_t)q | (uintptr_t)out | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) return -8;
    const int TQ = sg::ROWS / G;
    const long long tiles = (n_tok + TQ - 1) / TQ + n_items;          // an upper bound: every request may end a tile early
    if (tiles > 65535) return -8;
    CUtensorMap mk, mv;
    const uint64_t rows = (uint64_t)n_pages * page_size, kc = (uint64_t)nkv * hd, vc = (uint64_t)nkv * vd;
    int rc = tc::get_map(k_cache, rows, kc, kc, (uint32_t)page_size, &mk);
    if (rc) return rc;
    rc = tc::get_map(v_cache, rows, vc, vc, (uint32_t)page_size, &mv);
    if (rc) return rc;
    sg::Args a;
    a.q = (const __nv_bfloat16*)q; a.out = (__nv_bfloat16*)out;
    a.item_row_start = item_row_start; a.item_start_pos = item_start_pos; a.table = table; a.bias = bias; a.status = status;
    a.n_items = n_items; a.max_blocks = max_blocks; a.page_size = page_size; a.n_pages = n_pages; a.window = window; a.chunk = chunk;
    a.nh = nh; a.nkv = nkv; a.hd = hd; a.vd = vd; a.scale = scale;
    const dim3 grid(nkv, (unsigned)tiles);
    if (hd <= 64) return vd <= 64 ? sg::launch_prefill<1, 1>(mk, mv, a, grid, stream) : sg::launch_prefill<1, 2>(mk, mv, a, grid, stream);
    return vd <= 64 ? sg::launch_prefill<2, 1>(mk, mv, a, grid, stream) : sg::launch_prefill<2, 2>(mk, mv, a, grid, stream);
}

// bfloat16; hd and vd multiples of 16 up to 128, at most 8 query heads per kv head; else -8.  range: keys per CTA, a multiple of
// 64, counted from the query's first key; n_splits * range must cover the longest span of keys a query can see.  part_acc
// [n_tok, nh, n_splits, vd], part_ml [n_tok, nh, n_splits, 2].  fresh: the most tokens one request brings to this step (0: not known).
extern "C" int imparo_attention_sigmoid_split(const void* q, const void* k_cache, const void* v_cache, const int* positions,
                                              const int* item_of_token, const int* table, int max_blocks, int page_size, int n_pages,
                                              int window, int chunk, float scale, const float* bias, float* part_acc, float* part_ml,
                                              int n_tok, int nh, int nkv, int hd, int vd, int range, int n_splits, int fresh, int* status,
                                              cudaStream_t stream) {
    if (n_tok <= 0) return 0;
    if (nkv <= 0 || nh % nkv != 0) return -5;
    if (nh / nkv > 8 || hd < 16 || hd > 128 || hd % 16 || vd < 16 || vd > 128 || vd % 16) return -8;
    if (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) return -8;
    if (n_tok > 65535 || nkv > 65535 || range < 64 || range % 64 || n_splits < 1 || n_splits > 2048) return -2;
    long long span = (long long)max_blocks * page_size;
    if (window > 0 && window < span) span = window;
    if (chunk > 0 && chunk < span) span = chunk;
    if ((long long)range * n_splits < span) return -2;
    const dim3 grid(n_splits, nkv, n_tok);
#define IMPARO_SG(KW_, VW_) do { \
        constexpr size_t tiles = (size_t)2 * sg::DKEYS * ((KW_) + (VW_)) * 2, sums = (size_t)4 * 8 * (VW_) * 4; \
        constexpr size_t smem = tiles > sums ? tiles : sums; \
        static bool configured = false; \
        if (!configured) { \
            cudaError_t e = cudaFuncSetAttribute(sg::split_kernel<KW_, VW_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e; \
            configured = true; \
        } \
        launch(sg::split_kernel<KW_, VW_>, grid, dim3(sg::DT), smem, stream, (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, \
               (const __nv_bfloat16*)v_cache, positions, item_of_token, table, max_blocks, page_size, n_pages, window, chunk, scale, bias, \
               part_acc, part_ml, nh, nkv, hd, vd, range, n_splits, fresh, status); } while (0)
    if (hd <= 64) { if (vd <= 64) IMPARO_SG(64, 64); else IMPARO_SG(64, 128); }
    else { if (vd <= 64) IMPARO_SG(128, 64); else IMPARO_SG(128, 128); }
#undef IMPARO_SG
    IMPARO_CHECK_LAUNCH();
    return 0;
}
