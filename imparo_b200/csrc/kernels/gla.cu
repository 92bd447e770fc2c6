// Gated linear attention: a recurrence over a fixed-size state per request and head whose decay is one number per key channel
// and token,
//
//     alpha_t = sigmoid(z_t)^(1/tau),   z_t = W_2 l_t + b          (l_t: a few channels the input was brought down to)
//     S_t = diag(alpha_t) S_(t-1) + k_t v_t^T        S: [dim, vdim], S_0 = 0
//     o_t = S_t^T q_t,                               q_t already times q_scale
//
// for ragged batches: a request's rows are walked in order from what its slot holds, and the slot is written back at the end, so
// a prompt cut into portions, or decoded token by token, runs the same recurrence as the whole prompt.  Decays, their
// logarithms, the state and the sums are 32-bit; q, k, v and l are columns of products in the activations' dtype.
//
//  (1) gla_decay: log alpha = log sigmoid(z) / tau, [tokens, heads * dim] in 32-bit.
//  (2) gla_recurrent: up to four warps of one (request, head) per CTA.  A lane owns one column of S in registers (dim values;
//      beyond key size 64 two lanes share a column, each with half of the key channels); the rows' q, k, alpha and v pass
//      through shared memory in stages, q, k and alpha once for the CTA's warps.
//  (3) gla_step: the same for a step in which every request brings one row, with what stands around the recurrence in the
//      same kernel: the decay from l, and each head's norm, its weight and the silu gate on the way out.  A CTA owns a (request,
//      head) with all of its value columns.
//  (4) long portions in bfloat16 in chunks of 64 rows side by side, three launches.  With G_i the running sum of the log decays
//      inside a chunk (per key channel) the recurrence unrolls to
//          S_end = diag(exp(G_end)) S_in + sum_j (k_j * exp(G_end - G_j)) v_j^T
//          o_i   = S_in^T (q_i * exp(G_i)) + sum_(j<=i) [ sum_d q_i[d] k_j[d] exp(G_i[d] - G_j[d]) ] v_j
//        chunk_local: every chunk's own sum and exp(G_end); every exponent is <= 0
//        chunk_scan:  per request over its chunks in order: the state each chunk starts from; the slot at the end
//        chunk_out:   every chunk's outputs.  Scores as a product of q_i exp(G_i) and k_j exp(-G_j) when no channel of the chunk
//                     decays by more than e^-30 (the growing factor then stays far inside the range of 32-bit numbers), else
//                     pair by pair with exponents <= 0.  Where a CTA has all value columns of its head the norm, the weight and
//                     the gate follow in the same kernel.
//      The products run on tensor cores (mma.sync m16n8k16): whatever a decay has touched, the starting states and the scores
//      enter as the sum of a high and a low bfloat16 part (two or three products), so nothing of the recurrence is rounded to
//      8 bits; the state itself is only ever multiplied by its decay and added to in 32-bit.
#include "common.cuh"

namespace imparo {
namespace gla {

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// by the approximate exponential and logarithm: within 2e-7 of the above (a decay is the exponential of this over tau)
__device__ __forceinline__ float log_sigmoid_fast(float z) { return fminf(z, 0.f) - __logf(1.0f + __expf(-fabsf(z))); }

// ---- (1) ------------------------------------------------------------------------------------------------------
constexpr int DECAY_ROWS = 8;

template <typename T>
__global__ void __launch_bounds__(128)
decay_kernel(const T* __restrict__ low, size_t low_stride, const T* __restrict__ w2, const float* __restrict__ bias, float tau,
             float* __restrict__ out, int n_tok, int channels, int rank) {
    extern __shared__ float low_s[];                          // [DECAY_ROWS][rank]
    pdl_trigger();
    const int c = blockIdx.y * 128 + threadIdx.x;
    const int t0 = blockIdx.x * DECAY_ROWS, n = min(DECAY_ROWS, n_tok - t0);
    const float b = c < channels ? bias[c] : 0.f;
    pdl_wait();
    for (int i = threadIdx.x; i < n * rank; i += 128) low_s[i] = to_f32(low[(size_t)(t0 + i / rank) * low_stride + i % rank]);
    __syncthreads();
    if (c >= channels) return;
    float acc[DECAY_ROWS];
#pragma unroll
    for (int r = 0; r < DECAY_ROWS; ++r) acc[r] = 0.f;
    const T* wr = w2 + (size_t)c * rank;
    for (int k = 0; k < rank; ++k) {
        const float w = to_f32(wr[k]);
#pragma unroll
        for (int r = 0; r < DECAY_ROWS; ++r) acc[r] += r < n ? w * low_s[r * rank + k] : 0.f;
    }
#pragma unroll
    for (int r = 0; r < DECAY_ROWS; ++r)
        if (r < n) out[(size_t)(t0 + r) * channels + c] = log_sigmoid(acc[r] + b) / tau;
}

// ---- (2) ------------------------------------------------------------------------------------------------------
template <typename T>
struct Cols {
    const T* proj;          // rows of `stride` elements
    size_t stride;
    int q_off, k_off, v_off;
    const float* g;         // log decays [tokens, heads * dim]
    float q_scale;
};

template <int DMAX> struct Stage { static constexpr int ROWS = DMAX <= 64 ? 16 : 8; };

template <typename T, int DMAX, int NW, int SPLIT>
__global__ void __launch_bounds__(NW * 32)
recurrent_kernel(Cols<T> c, float* __restrict__ state, const int* __restrict__ item_row_start, const int* __restrict__ item_slot,
                 int n_slots, float* __restrict__ out, int heads, int dim, int vdim, int* status) {
    constexpr int ST = Stage<DMAX>::ROWS, DL = DMAX / SPLIT, WCOLS = 32 / SPLIT, THREADS = NW * 32;
    __shared__ __align__(16) float q_s[ST][DMAX], k_s[ST][DMAX], a_s[ST][DMAX], v_s[ST][NW * WCOLS];
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int item = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * NW * WCOLS;
    const int my = warp * WCOLS + lane % WCOLS, col = v0 + my, dofs = (lane / WCOLS) * DL;
    const int r0 = item_row_start[item], r1 = item_row_start[item + 1];
    const int slot = item_slot[item];
    pdl_wait();
    if (slot < 0 || slot >= n_slots) {
        if (tid == 0 && blockIdx.z == 0) report(status, IMPARO_ST_SLOT_RANGE, 91, item, slot);
        return;
    }
    const bool live = col < vdim;
    const int vcols = min(NW * WCOLS, vdim - v0);
    float* sp = state + (((size_t)slot * heads + h) * dim) * vdim + col;
    float S[DL];
#pragma unroll
    for (int d = 0; d < DL; ++d) S[d] = (live && dofs + d < dim) ? sp[(size_t)(dofs + d) * vdim] : 0.f;
    for (int base = r0; base < r1; base += ST) {
        const int n = min(ST, r1 - base);
        __syncthreads();
        for (int i = tid; i < n * DMAX; i += THREADS) {
            const int r = i / DMAX, d = i % DMAX;
            float q = 0.f, k = 0.f, a = 0.f;
            if (d < dim) {
                const T* row = c.proj + (size_t)(base + r) * c.stride + (size_t)h * dim + d;
                q = to_f32(row[c.q_off]) * c.q_scale;
                k = to_f32(row[c.k_off]);
                a = expf(c.g[((size_t)(base + r) * heads + h) * dim + d]);
            }
            q_s[r][d] = q; k_s[r][d] = k; a_s[r][d] = a;
        }
        for (int i = tid; i < n * NW * WCOLS; i += THREADS) {
            const int r = i / (NW * WCOLS), p = i % (NW * WCOLS);
            v_s[r][p] = p < vcols ? to_f32(c.proj[(size_t)(base + r) * c.stride + c.v_off + (size_t)h * vdim + v0 + p]) : 0.f;
        }
        __syncthreads();
        for (int r = 0; r < n; ++r) {
            const float vv = v_s[r][my];
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
            for (int d = 0; d < DL; d += 4) {
                const float4 a4 = *reinterpret_cast<const float4*>(&a_s[r][dofs + d]);
                const float4 k4 = *reinterpret_cast<const float4*>(&k_s[r][dofs + d]);
                const float4 q4 = *reinterpret_cast<const float4*>(&q_s[r][dofs + d]);
                S[d] = a4.x * S[d] + k4.x * vv;             o0 += S[d] * q4.x;
                S[d + 1] = a4.y * S[d + 1] + k4.y * vv;     o1 += S[d + 1] * q4.y;
                S[d + 2] = a4.z * S[d + 2] + k4.z * vv;     o2 += S[d + 2] * q4.z;
                S[d + 3] = a4.w * S[d + 3] + k4.w * vv;     o3 += S[d + 3] * q4.w;
            }
            float o = (o0 + o1) + (o2 + o3);
            if (SPLIT == 2) o += __shfl_xor_sync(0xffffffffu, o, 16);              // the other half of the key channels
            if (live && lane < WCOLS) out[((size_t)(base + r) * heads + h) * vdim + col] = o;
        }
    }
    if (live) {
#pragma unroll
        for (int d = 0; d < DL; ++d) if (dofs + d < dim) sp[(size_t)(dofs + d) * vdim] = S[d];
    }
}

template <typename T, int DMAX>
static int launch_recurrent(const Cols<T>& c, float* state, const int* item_row_start, const int* item_slot, int n_slots,
                            int n_items, float* out, int heads, int dim, int vdim, int* status, cudaStream_t stream) {
    constexpr int SPLIT = DMAX > 64 ? 2 : 1, WCOLS = 32 / SPLIT;
    const int blocks = (vdim + WCOLS - 1) / WCOLS;             // warps a head's value columns fill
#define IMPARO_GR(NW_) launch(recurrent_kernel<T, DMAX, NW_, SPLIT>, dim3(n_items, heads, (blocks + NW_ - 1) / NW_), dim3(NW_ * 32), 0, \
        stream, c, state, item_row_start, item_slot, n_slots, out, heads, dim, vdim, status)
    if (blocks >= 3) IMPARO_GR(4);
    else if (blocks == 2) IMPARO_GR(2);
    else IMPARO_GR(1);
#undef IMPARO_GR
    IMPARO_CHECK_LAUNCH();
    return 0;
}

// ---- (3) ------------------------------------------------------------------------------------------------------
// Warps of 32 / SPLIT value columns each cover the head's; SPLIT lanes share a column, each with its stretch of the key channels.
template <typename T, int DMAX, int SPLIT>
__global__ void __launch_bounds__(512)
step_kernel(Cols<T> c, int l_off, const T* __restrict__ w2, const float* __restrict__ bias, float tau, int rank, int g_off,
            const float* __restrict__ w_norm, float eps, float* __restrict__ state, const int* __restrict__ item_row_start,
            const int* __restrict__ item_slot, int n_slots, T* __restrict__ out, int heads, int dim, int vdim, int* status) {
    constexpr int DL = DMAX / SPLIT, WCOLS = 32 / SPLIT;
    __shared__ __align__(16) float q_s[DMAX], k_s[DMAX], a_s[DMAX];
    __shared__ float scratch[33];
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int item = blockIdx.x, h = blockIdx.y;
    const int col = warp * WCOLS + lane % WCOLS, dofs = (lane / WCOLS) * DL;
    const int r = item_row_start[item];
    const int slot = item_slot[item];
    const bool live = col < vdim;
    const float wn = live ? w_norm[col] : 0.f;
    pdl_wait();
    if (slot < 0 || slot >= n_slots) {                         // (uniform over the CTA)
        if (tid == 0) report(status, IMPARO_ST_SLOT_RANGE, 92, item, slot);
        return;
    }
    float* sp = state + (((size_t)slot * heads + h) * dim) * vdim + col;
    const T* row = c.proj + (size_t)r * c.stride;
    float S[DL];
#pragma unroll
    for (int d = 0; d < DL; ++d) S[d] = (live && dofs + d < dim) ? sp[(size_t)(dofs + d) * vdim] : 0.f;
    const float vv = live ? to_f32(row[c.v_off + (size_t)h * vdim + col]) : 0.f;
    const float gate = live ? to_f32(row[g_off + (size_t)h * vdim + col]) : 0.f;
    for (int d = tid; d < DMAX; d += blockDim.x) {
        float q = 0.f, k = 0.f, a = 0.f;
        if (d < dim) {
            q = to_f32(row[c.q_off + (size_t)h * dim + d]) * c.q_scale;
            k = to_f32(row[c.k_off + (size_t)h * dim + d]);
            const T* wr = w2 + ((size_t)h * dim + d) * rank;
            float z = 0.f;
            for (int i = 0; i < rank; ++i) z += to_f32(wr[i]) * to_f32(row[l_off + i]);
            a = expf(log_sigmoid(z + bias[(size_t)h * dim + d]) / tau);
        }
        q_s[d] = q; k_s[d] = k; a_s[d] = a;
    }
    __syncthreads();
    float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
    for (int d = 0; d < DL; d += 4) {
        const float4 a4 = *reinterpret_cast<const float4*>(&a_s[dofs + d]);
        const float4 k4 = *reinterpret_cast<const float4*>(&k_s[dofs + d]);
        const float4 q4 = *reinterpret_cast<const float4*>(&q_s[dofs + d]);
        S[d] = a4.x * S[d] + k4.x * vv;             o0 += S[d] * q4.x;
        S[d + 1] = a4.y * S[d + 1] + k4.y * vv;     o1 += S[d + 1] * q4.y;
        S[d + 2] = a4.z * S[d + 2] + k4.z * vv;     o2 += S[d + 2] * q4.z;
        S[d + 3] = a4.w * S[d + 3] + k4.w * vv;     o3 += S[d + 3] * q4.w;
    }
    if (live) {
#pragma unroll
        for (int d = 0; d < DL; ++d) if (dofs + d < dim) sp[(size_t)(dofs + d) * vdim] = S[d];
    }
    float o = (o0 + o1) + (o2 + o3);
#pragma unroll
    for (int s = WCOLS; s < 32; s <<= 1) o += __shfl_xor_sync(0xffffffffu, o, s);      // the other stretches of the key channels
    const float ss = block_sum((live && lane < WCOLS) ? o * o : 0.f, scratch);
    if (live && lane < WCOLS) {
        const float y = o * (1.0f / sqrtf(ss / (float)vdim + eps)) * wn * silu(gate);
        out[((size_t)r * heads + h) * vdim + col] = from_f32<T>(y);
    }
}

// ---- (4) ------------------------------------------------------------------------------------------------------
constexpr int C = 64;               // rows per chunk
constexpr int PAD = 8;              // elements between a tile's rows: eight rows of an ldmatrix fall into distinct banks
constexpr int CT = 256;             // threads: eight warps of 16 value columns each
constexpr int CCOLS = 128;          // value columns of a CTA
constexpr float FAST_DECAY = 30.f;
using bf16 = __nv_bfloat16;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// a pair of 32-bit numbers as high and low bfloat16 pairs
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

struct Chunks {
    const bf16* proj;
    size_t stride;
    int q_off, k_off, v_off, g_off;
    float* g;                   // log decays [tokens, heads * dim]: read, or (DECAY) made and written by chunk_local
    int l_off, rank;            // DECAY: the decay's inner columns, w2 [heads * dim, rank], bias [heads * dim], tau
    const bf16* w2;
    const float* bias;
    float tau;
    float q_scale;
    const int* item_row_start;
    int n_items;
    float* state;               // [chunks, heads, dim, vdim]
    float* decay;               // [chunks, heads, dim]
    int heads, dim, vdim;
};

// the chunks of all requests of the launch are numbered in order; the grid's x extent is an upper bound of their number
__device__ __forceinline__ bool find_chunk(const int* __restrict__ item_row_start, int n_items, int g, int& r_begin, int& r_end) {
    int base = 0;
    for (int i = 0; i < n_items; ++i) {
        const int r0 = item_row_start[i], r1 = item_row_start[i + 1];
        const int nc = (r1 - r0 + C - 1) / C;
        if (g < base + nc) {
            r_begin = r0 + (g - base) * C;
            r_end = min(r_begin + C, r1);
            return true;
        }
        base += nc;
    }
    return false;
}

// A thread's share of the chunk's log decays.  Channel pairs are shared out over dim / 2 threads, the chunk's rows over `segs`
// segments of `per` <= PER rows, which the thread keeps in registers (x; rows the chunk does not have are 0).
constexpr int PER = 16;
struct Walk {
    int pair, seg, segs, per, r0;       // r0: the segment's first row; pair < 0: the thread has none
    float2 x[PER], start, total;        // start: the sum of the segments before; total: the chunk's
};
__device__ __forceinline__ void walk_share(Walk& w, int dim) {
    const int pairs = dim / 2;
    w.segs = min(C, CT / pairs);
    w.per = (C + w.segs - 1) / w.segs;
    w.seg = threadIdx.x / pairs;
    w.pair = w.seg < w.segs ? (int)threadIdx.x % pairs : -1;
    w.r0 = w.seg * w.per;
}
// x -> start and total; all threads of the CTA call it
__device__ __forceinline__ void walk_sums(Walk& w, int dim, float* seg_sum /* [segs][dim] */) {
    if (w.pair >= 0) {
        float2 s = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < PER; ++i) { s.x += w.x[i].x; s.y += w.x[i].y; }
        *reinterpret_cast<float2*>(seg_sum + (size_t)w.seg * dim + 2 * w.pair) = s;
    }
    __syncthreads();
    w.start = w.total = make_float2(0.f, 0.f);
    if (w.pair >= 0) {
        for (int i = 0; i < w.segs; ++i) {
            const float2 x = *reinterpret_cast<const float2*>(seg_sum + (size_t)i * dim + 2 * w.pair);
            if (i < w.seg) { w.start.x += x.x; w.start.y += x.y; }
            w.total.x += x.x; w.total.y += x.y;
        }
    }
}

// rows [0, n) of the CTA's value columns -> v_s [C][ldv], the rest zero
__device__ __forceinline__ void stage_values(const bf16* __restrict__ src, size_t stride, int n, int vcols, bf16* __restrict__ v_s, int ldv) {
    const int vecs = vcols / 8;
    for (int i = threadIdx.x; i < C * vecs; i += CT) {
        const int r = i / vecs, c = (i - r * vecs) * 8;
        uint4 x = make_uint4(0u, 0u, 0u, 0u);
        if (r < n) x = *reinterpret_cast<const uint4*>(src + (size_t)r * stride + c);
        *reinterpret_cast<uint4*>(v_s + (size_t)r * ldv + c) = x;
    }
}

// DECAY: the log decays are made here from the inner columns (rank <= MAX_RANK) and left in a.g for chunk_out.
constexpr int MAX_RANK = 32;

template <bool DECAY>
__global__ void __launch_bounds__(CT, 3)
chunk_local_kernel(const Chunks a) {
    extern __shared__ __align__(16) unsigned char gla_smem[];
    pdl_trigger();
    const int g = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * CCOLS;
    int r_begin, r_end;
    const bool found = find_chunk(a.item_row_start, a.n_items, g, r_begin, r_end);
    const int dim = a.dim, vcols = min(CCOLS, a.vdim - v0);
    const int ldk = dim + PAD, ldv = vcols + PAD;
    bf16* k_hi = reinterpret_cast<bf16*>(gla_smem);
    bf16* k_lo = k_hi + C * ldk;
    bf16* v_s = k_lo + C * ldk;
    float* seg_sum = reinterpret_cast<float*>(v_s + C * ldv);
    float* w2_s = seg_sum + (size_t)min(C, 2 * CT / dim) * dim;          // [rank][dim]
    Walk w;
    walk_share(w, dim);
    const int per4 = (w.per + 3) & ~3, ldl = w.segs * per4;               // a segment's rows start on 16 bytes
    float* low_s = w2_s + (size_t)a.rank * dim;                           // [rank][segs][per4], at most 2 * C per inner channel
    float2 bias2 = make_float2(0.f, 0.f);
    if (DECAY) {
        const bf16* src = a.w2 + (size_t)h * dim * a.rank;
        for (int e = threadIdx.x; e < dim * a.rank; e += CT) w2_s[(e % a.rank) * dim + e / a.rank] = to_f32(src[e]);
        if (w.pair >= 0) bias2 = make_float2(a.bias[h * dim + 2 * w.pair], a.bias[h * dim + 2 * w.pair + 1]);
    }
    pdl_wait();
    if (!found) return;
    const int n = r_end - r_begin;
    stage_values(a.proj + (size_t)r_begin * a.stride + a.v_off + (size_t)h * a.vdim + v0, a.stride, n, vcols, v_s, ldv);
    const size_t gs = (size_t)a.heads * dim;
    float* gp = a.g + (size_t)r_begin * gs + (size_t)h * dim + 2 * w.pair;
    if (DECAY) {
        for (int e = threadIdx.x; e < C * a.rank; e += CT) {
            const int r = e / a.rank, k = e - r * a.rank;
            low_s[k * ldl + r / w.per * per4 + r % w.per] = r < n ? to_f32(a.proj[(size_t)(r_begin + r) * a.stride + a.l_off + k]) : 0.f;
        }
        __syncthreads();
        if (w.pair >= 0) {
            const float inv_tau = 1.0f / a.tau;
#pragma unroll
            for (int i = 0; i < PER; ++i) w.x[i] = bias2;
            for (int k = 0; k < a.rank; ++k) {
                const float2 c = *reinterpret_cast<const float2*>(w2_s + (size_t)k * dim + 2 * w.pair);
                const float* l = low_s + k * ldl + w.seg * per4;
#pragma unroll
                for (int i = 0; i < PER; i += 4) {
                    if (i < per4) {                            // (places past the segment's rows hold anything; their sums are dropped)
                        const float4 x = *reinterpret_cast<const float4*>(l + i);
                        w.x[i].x += c.x * x.x; w.x[i].y += c.y * x.x;
                        w.x[i + 1].x += c.x * x.y; w.x[i + 1].y += c.y * x.y;
                        w.x[i + 2].x += c.x * x.z; w.x[i + 2].y += c.y * x.z;
                        w.x[i + 3].x += c.x * x.w; w.x[i + 3].y += c.y * x.w;
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int r = w.r0 + i;
                if (i < w.per && r < n) {
                    w.x[i] = make_float2(log_sigmoid_fast(w.x[i].x) * inv_tau, log_sigmoid_fast(w.x[i].y) * inv_tau);
                    *reinterpret_cast<float2*>(gp + (size_t)r * gs) = w.x[i];
                } else {
                    w.x[i] = make_float2(0.f, 0.f);
                }
            }
        }
    } else if (w.pair >= 0) {
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = w.r0 + i;
            w.x[i] = (i < w.per && r < n) ? *reinterpret_cast<const float2*>(gp + (size_t)r * gs) : make_float2(0.f, 0.f);
        }
    }
    __nv_bfloat162 kr[PER];
    if (w.pair >= 0) {
        const bf16* kp = a.proj + (size_t)r_begin * a.stride + a.k_off + (size_t)h * dim + 2 * w.pair;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = w.r0 + i;
            kr[i] = __floats2bfloat162_rn(0.f, 0.f);
            if (i < w.per && r < n) kr[i] = *reinterpret_cast<const __nv_bfloat162*>(kp + (size_t)r * a.stride);
        }
    }
    walk_sums(w, dim, seg_sum);
    if (w.pair >= 0) {
        float2 G = w.start;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = w.r0 + i;
            if (i < w.per && r < C) {                         // (rows the chunk does not have: keys of zero)
                G.x += w.x[i].x; G.y += w.x[i].y;
                const float2 k = __bfloat1622float2(kr[i]);
                uint32_t hi, lo;
                split2(k.x * __expf(w.total.x - G.x), k.y * __expf(w.total.y - G.y), hi, lo);
                *reinterpret_cast<uint32_t*>(k_hi + (size_t)r * ldk + 2 * w.pair) = hi;
                *reinterpret_cast<uint32_t*>(k_lo + (size_t)r * ldk + 2 * w.pair) = lo;
            }
        }
        if (w.seg == 0 && blockIdx.z == 0)
            *reinterpret_cast<float2*>(a.decay + ((size_t)g * a.heads + h) * dim + 2 * w.pair) = make_float2(__expf(w.total.x), __expf(w.total.y));
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n0 = warp * 16;
    if (n0 >= vcols) return;
    const int mi = lane >> 3, rin = lane & 7, gq = lane >> 2, tg = lane & 3;
    const int ksteps = (n + 15) / 16;
    float* dst = a.state + (((size_t)g * a.heads + h) * dim) * a.vdim + v0 + n0;
    uint32_t b[C / 16][4];
#pragma unroll
    for (int kk = 0; kk < C / 16; ++kk)                       // values: (k = row j, n = column), stored [j][n]
        if (kk < ksteps) ldmatrix4_trans(b[kk], v_s + (size_t)(kk * 16 + (mi & 1) * 8 + rin) * ldv + n0 + (mi >> 1) * 8);
    for (int mt = 0; mt < dim / 16; ++mt) {
        float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int kk = 0; kk < C / 16; ++kk) {
            if (kk < ksteps) {
                // keys: (m = channel, k = row j), stored [j][channel]: matrices (m0, k0), (m8, k0), (m0, k8), (m8, k8)
                uint32_t ah[4], al[4];
                const size_t off = (size_t)(kk * 16 + (mi >> 1) * 8 + rin) * ldk + mt * 16 + (mi & 1) * 8;
                ldmatrix4_trans(ah, k_hi + off);
                ldmatrix4_trans(al, k_lo + off);
                mma(c0, ah, b[kk][0], b[kk][1]); mma(c1, ah, b[kk][2], b[kk][3]);
                mma(c0, al, b[kk][0], b[kk][1]); mma(c1, al, b[kk][2], b[kk][3]);
            }
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            float* row = dst + (size_t)(mt * 16 + gq + half * 8) * a.vdim + 2 * tg;
            *reinterpret_cast<float2*>(row) = make_float2(c0[2 * half], c0[2 * half + 1]);
            *reinterpret_cast<float2*>(row + 8) = make_float2(c1[2 * half], c1[2 * half + 1]);
        }
    }
}

// grid (requests, heads, ceil(dim * vdim / 4 / 256)): four neighbouring state entries (of one key channel) per thread
__global__ void __launch_bounds__(256)
chunk_scan_kernel(const Chunks a, float* __restrict__ slots, const int* __restrict__ item_slot, int n_slots, int* status) {
    pdl_trigger();
    const int item = blockIdx.x, h = blockIdx.y;
    const int per_head = a.dim * a.vdim;
    const int e = (blockIdx.z * 256 + threadIdx.x) * 4;
    int first = 0;
    for (int i = 0; i < item; ++i) first += (a.item_row_start[i + 1] - a.item_row_start[i] + C - 1) / C;
    const int nc = (a.item_row_start[item + 1] - a.item_row_start[item] + C - 1) / C;
    const int slot = item_slot[item];
    pdl_wait();
    if (slot < 0 || slot >= n_slots) {
        if (threadIdx.x == 0 && blockIdx.z == 0) report(status, IMPARO_ST_SLOT_RANGE, 93, item, slot);
        return;
    }
    if (e >= per_head) return;
    float4* sp = reinterpret_cast<float4*>(slots + ((size_t)slot * a.heads + h) * per_head + e);
    float4 s = *sp;
    float* cp = a.state + ((size_t)first * a.heads + h) * per_head + e;
    const float* dp = a.decay + ((size_t)first * a.heads + h) * a.dim + e / a.vdim;
    const size_t cs = (size_t)a.heads * per_head, ds = (size_t)a.heads * a.dim;
    constexpr int U = 8;
    for (int c0 = 0; c0 < nc; c0 += U) {                      // eight chunks' loads at once, then the chain
        float4 loc[U];
        float dec[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u < nc) {
                loc[u] = __ldcg(reinterpret_cast<const float4*>(cp + (size_t)(c0 + u) * cs));
                dec[u] = __ldcg(dp + (size_t)(c0 + u) * ds);
            }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u < nc) {
                *reinterpret_cast<float4*>(cp + (size_t)(c0 + u) * cs) = s;        // the state this chunk starts from
                s.x = dec[u] * s.x + loc[u].x; s.y = dec[u] * s.y + loc[u].y;
                s.z = dec[u] * s.z + loc[u].z; s.w = dec[u] * s.w + loc[u].w;
            }
        }
    }
    *sp = s;
}

// NORM: the CTA has all value columns of its head; y = bfloat16 of the normed, weighted, gated output.  Else o in 32-bit.
template <bool NORM>
__global__ void __launch_bounds__(CT)
chunk_out_kernel(const Chunks a, const float* __restrict__ w_norm, float eps, float* __restrict__ o_out, bf16* __restrict__ y_out) {
    extern __shared__ __align__(16) unsigned char gla_smem[];
    __shared__ float row_ss[CT / 32][C];
    pdl_trigger();
    const int g = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * CCOLS;
    int r_begin, r_end;
    const bool found = find_chunk(a.item_row_start, a.n_items, g, r_begin, r_end);
    pdl_wait();
    if (!found) return;
    const int n = r_end - r_begin, dim = a.dim, vcols = min(CCOLS, a.vdim - v0);
    const int ldq = dim + PAD, ldv = vcols + PAD;
    constexpr int lda = C + PAD;
    bf16* q_hi = reinterpret_cast<bf16*>(gla_smem);           // q exp(G)
    bf16* q_lo = q_hi + C * ldq;
    bf16* k_hi = q_lo + C * ldq;                              // k exp(-G); afterwards the scores
    bf16* k_lo = k_hi + C * (ldq > lda ? ldq : lda);
    bf16* v_s = k_lo + C * (ldq > lda ? ldq : lda);
    float* seg_sum = reinterpret_cast<float*>(v_s + C * ldv);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n0 = warp * 16;
    const int mi = lane >> 3, rin = lane & 7, gq = lane >> 2, tg = lane & 3;
    const bool busy = n0 < vcols;
    const float* S0 = a.state + (((size_t)g * a.heads + h) * dim) * a.vdim + v0 + n0;
    stage_values(a.proj + (size_t)r_begin * a.stride + a.v_off + (size_t)h * a.vdim + v0, a.stride, n, vcols, v_s, ldv);
    const size_t gs = (size_t)a.heads * dim;
    Walk w;
    walk_share(w, dim);
    __nv_bfloat162 qr[PER], kr[PER];
    if (w.pair >= 0) {                                        // everything the thread needs of its rows, requested at once
        const bf16* row = a.proj + (size_t)r_begin * a.stride + (size_t)h * dim + 2 * w.pair;
        const float* gp = a.g + (size_t)r_begin * gs + (size_t)h * dim + 2 * w.pair;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = w.r0 + i;
            w.x[i] = make_float2(0.f, 0.f);
            qr[i] = kr[i] = __floats2bfloat162_rn(0.f, 0.f);
            if (i < w.per && r < n) {
                w.x[i] = *reinterpret_cast<const float2*>(gp + (size_t)r * gs);
                qr[i] = *reinterpret_cast<const __nv_bfloat162*>(row + (size_t)r * a.stride + a.q_off);
                kr[i] = *reinterpret_cast<const __nv_bfloat162*>(row + (size_t)r * a.stride + a.k_off);
            }
        }
    }
    float s_next[8];                                          // the starting state's entries of the next 16 channels
    auto load_state = [&](int kk) {
#pragma unroll
        for (int e = 0; e < 8; ++e)
            s_next[e] = __ldcg(S0 + (size_t)(kk * 16 + ((e >> 1) & 1) * 8 + 2 * tg + (e & 1)) * a.vdim + (e >> 2) * 8 + gq);
    };
    if (busy) load_state(0);
    walk_sums(w, dim, seg_sum);
    float* G_s = reinterpret_cast<float*>(k_hi);              // the slow form keeps the running sums here instead
    const int slow = __syncthreads_or(w.pair >= 0 && (w.total.x < -FAST_DECAY || w.total.y < -FAST_DECAY));
    if (w.pair >= 0) {
        float2 G = w.start;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int r = w.r0 + i;
            if (i < w.per && r < C) {                         // (rows the chunk does not have: queries and keys of zero)
                G.x += w.x[i].x; G.y += w.x[i].y;
                const float2 q = __bfloat1622float2(qr[i]);
                uint32_t hi, lo;
                const size_t at = (size_t)r * ldq + 2 * w.pair;
                split2(q.x * a.q_scale * __expf(G.x), q.y * a.q_scale * __expf(G.y), hi, lo);
                *reinterpret_cast<uint32_t*>(q_hi + at) = hi;
                *reinterpret_cast<uint32_t*>(q_lo + at) = lo;
                if (slow) {
                    *reinterpret_cast<float2*>(G_s + (size_t)r * dim + 2 * w.pair) = G;
                } else {
                    const float2 k = __bfloat1622float2(kr[i]);
                    split2(k.x * __expf(-G.x), k.y * __expf(-G.y), hi, lo);
                    *reinterpret_cast<uint32_t*>(k_hi + at) = hi;
                    *reinterpret_cast<uint32_t*>(k_lo + at) = lo;
                }
            }
        }
    }
    __syncthreads();
    bf16* a_hi = k_hi;
    bf16* a_lo = k_lo;
    if (!slow) {
        // scores of the 16 x 16 tiles on and below the diagonal, (0,0) (1,0) (1,1) (2,0) ...; a warp takes tiles warp and warp + 8
        float c[2][2][4];
#pragma unroll
        for (int s = 0; s < 2; ++s) {
            const int t = warp + s * 8;
            int it = 0, jt = t;
            while (jt > it) { jt -= it + 1; ++it; }
#pragma unroll
            for (int e = 0; e < 4; ++e) c[s][0][e] = c[s][1][e] = 0.f;
            if (t < 10) {
                for (int kk = 0; kk < dim / 16; ++kk) {
                    uint32_t ah[4], al[4], bh[4], bl[4];
                    const size_t qo = (size_t)(it * 16 + (mi & 1) * 8 + rin) * ldq + kk * 16 + (mi >> 1) * 8;
                    const size_t ko = (size_t)(jt * 16 + (mi >> 1) * 8 + rin) * ldq + kk * 16 + (mi & 1) * 8;
                    ldmatrix4(ah, q_hi + qo); ldmatrix4(al, q_lo + qo);
                    ldmatrix4(bh, k_hi + ko); ldmatrix4(bl, k_lo + ko);
                    mma(c[s][0], ah, bh[0], bh[1]); mma(c[s][1], ah, bh[2], bh[3]);
                    mma(c[s][0], ah, bl[0], bl[1]); mma(c[s][1], ah, bl[2], bl[3]);
                    mma(c[s][0], al, bh[0], bh[1]); mma(c[s][1], al, bh[2], bh[3]);
                }
            }
        }
        __syncthreads();                                      // the keys have been read: the scores take their place
#pragma unroll
        for (int s = 0; s < 2; ++s) {
            const int t = warp + s * 8;
            int it = 0, jt = t;
            while (jt > it) { jt -= it + 1; ++it; }
            if (t < 10) {
#pragma unroll
                for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        const int i = it * 16 + gq + half * 8, j = jt * 16 + nt * 8 + 2 * tg;
                        uint32_t hi, lo;
                        split2(j <= i ? c[s][nt][2 * half] : 0.f, j + 1 <= i ? c[s][nt][2 * half + 1] : 0.f, hi, lo);
                        *reinterpret_cast<uint32_t*>(a_hi + (size_t)i * lda + j) = hi;
                        *reinterpret_cast<uint32_t*>(a_lo + (size_t)i * lda + j) = lo;
                    }
            }
        }
    } else {
        // some channel decays too far for factors that grow: every pair's exponents by themselves.  A warp takes eight rows i, a lane
        // two columns j of each; the sums wait in registers until every running sum has been read.
        float sums[C / 8][2];
#pragma unroll
        for (int k = 0; k < C / 8; ++k) {
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int i = warp + 8 * k, j = lane + 32 * u;
                float sum = 0.f;
                if (i < n && j <= i) {
                    const bf16* qr = a.proj + (size_t)(r_begin + i) * a.stride + a.q_off + (size_t)h * dim;
                    const bf16* kr = a.proj + (size_t)(r_begin + j) * a.stride + a.k_off + (size_t)h * dim;
                    const float* Gi = G_s + (size_t)i * dim;
                    const float* Gj = G_s + (size_t)j * dim;
                    for (int d = 0; d < dim; ++d) sum += to_f32(qr[d]) * to_f32(kr[d]) * __expf(Gi[d] - Gj[d]);
                }
                sums[k][u] = sum * a.q_scale;
            }
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < C / 8; ++k)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const size_t at = (size_t)(warp + 8 * k) * lda + lane + 32 * u;
                const bf16 hi = __float2bfloat16_rn(sums[k][u]);
                a_hi[at] = hi;
                a_lo[at] = __float2bfloat16_rn(sums[k][u] - __bfloat162float(hi));
            }
    }
    __syncthreads();
    float o[4][2][4];                                         // four 16-row tiles x this warp's 16 columns
#pragma unroll
    for (int it = 0; it < 4; ++it)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[it][0][e] = o[it][1][e] = 0.f;
    if (busy) {
        for (int kk = 0; kk < dim / 16; ++kk) {               // the state the chunk starts from
            uint32_t bh[4], bl[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) split2(s_next[2 * e], s_next[2 * e + 1], bh[e], bl[e]);
            if (kk + 1 < dim / 16) load_state(kk + 1);
#pragma unroll
            for (int it = 0; it < 4; ++it) {
                uint32_t ah[4], al[4];
                const size_t qo = (size_t)(it * 16 + (mi & 1) * 8 + rin) * ldq + kk * 16 + (mi >> 1) * 8;
                ldmatrix4(ah, q_hi + qo); ldmatrix4(al, q_lo + qo);
                mma(o[it][0], ah, bh[0], bh[1]); mma(o[it][1], ah, bh[2], bh[3]);
                mma(o[it][0], ah, bl[0], bl[1]); mma(o[it][1], ah, bl[2], bl[3]);
                mma(o[it][0], al, bh[0], bh[1]); mma(o[it][1], al, bh[2], bh[3]);
            }
        }
#pragma unroll
        for (int jj = 0; jj < 4; ++jj) {                      // the chunk's own rows up to the diagonal
            uint32_t b[4];
            ldmatrix4_trans(b, v_s + (size_t)(jj * 16 + (mi & 1) * 8 + rin) * ldv + n0 + (mi >> 1) * 8);
#pragma unroll
            for (int it = jj; it < 4; ++it) {
                uint32_t ah[4], al[4];
                const size_t ao = (size_t)(it * 16 + (mi & 1) * 8 + rin) * lda + jj * 16 + (mi >> 1) * 8;
                ldmatrix4(ah, a_hi + ao); ldmatrix4(al, a_lo + ao);
                mma(o[it][0], ah, b[0], b[1]); mma(o[it][1], ah, b[2], b[3]);
                mma(o[it][0], al, b[0], b[1]); mma(o[it][1], al, b[2], b[3]);
            }
        }
    }
    if (!NORM) {
        if (!busy) return;
#pragma unroll
        for (int it = 0; it < 4; ++it)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int r = it * 16 + gq + half * 8;
                if (r < n) {
                    float* dst = o_out + ((size_t)(r_begin + r) * a.heads + h) * a.vdim + v0 + n0 + 2 * tg;
                    *reinterpret_cast<float2*>(dst) = make_float2(o[it][0][2 * half], o[it][0][2 * half + 1]);
                    *reinterpret_cast<float2*>(dst + 8) = make_float2(o[it][1][2 * half], o[it][1][2 * half + 1]);
                }
            }
        return;
    }
    // each row's sum of squares over the head's columns: four lanes of a warp, then the warps in order
#pragma unroll
    for (int it = 0; it < 4; ++it)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            float ss = o[it][0][2 * half] * o[it][0][2 * half] + o[it][0][2 * half + 1] * o[it][0][2 * half + 1] +
                       o[it][1][2 * half] * o[it][1][2 * half] + o[it][1][2 * half + 1] * o[it][1][2 * half + 1];
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            if (tg == 0) row_ss[warp][it * 16 + gq + half * 8] = ss;
        }
    __syncthreads();
    if (!busy) return;
    const int warps = (vcols + 15) / 16;
#pragma unroll
    for (int it = 0; it < 4; ++it)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = it * 16 + gq + half * 8;
            if (r >= n) continue;
            float ss = 0.f;
            for (int i = 0; i < warps; ++i) ss += row_ss[i][r];
            const float scale = 1.0f / sqrtf(ss / (float)a.vdim + eps);
            const bf16* gate = a.proj + (size_t)(r_begin + r) * a.stride + a.g_off + (size_t)h * a.vdim + n0 + 2 * tg;
            bf16* dst = y_out + ((size_t)(r_begin + r) * a.heads + h) * a.vdim + n0 + 2 * tg;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + nt * 8));
                const float2 wv = *reinterpret_cast<const float2*>(w_norm + n0 + nt * 8 + 2 * tg);
                const float y0 = o[it][nt][2 * half] * scale * wv.x * silu_bf16(z.x), y1 = o[it][nt][2 * half + 1] * scale * wv.y * silu_bf16(z.y);
                *reinterpret_cast<__nv_bfloat162*>(dst + nt * 8) = __floats2bfloat162_rn(y0, y1);
            }
        }
}

static size_t local_smem(int dim, int vcols, int rank) {
    return (size_t)rank * (dim + 2 * C) * 4 + (size_t)C * (2 * (dim + PAD) + (vcols + PAD)) * 2 + (size_t)(2 * CT / dim < C ? 2 * CT / dim : C) * dim * 4;
}
static size_t out_smem(int dim, int vcols) {
    const int ldk = dim + PAD > C + PAD ? dim + PAD : C + PAD;
    return (size_t)C * (2 * (dim + PAD) + 2 * ldk + (vcols + PAD)) * 2 + (size_t)(2 * CT / dim < C ? 2 * CT / dim : C) * dim * 4;
}

}  // namespace gla
}  // namespace imparo

using namespace imparo;

// low: rows of low_stride elements (rank used); w2 [channels, rank] in low's dtype; bias float32 [channels]; out float32
// [n_tok, channels] = log sigmoid(w2 low + bias) / tau.
extern "C" int imparo_gla_decay(const void* low, long long low_stride, int dtype, const void* w2, const float* bias, float tau,
                                float* out, int n_tok, int channels, int rank, cudaStream_t stream) {
    if (n_tok <= 0) return 0;
    if (channels < 1 || rank < 1 || rank > 1024 || low_stride < rank || !(tau > 0.f)) return -2;
    const dim3 grid((n_tok + gla::DECAY_ROWS - 1) / gla::DECAY_ROWS, (channels + 127) / 128);
    const size_t smem = (size_t)gla::DECAY_ROWS * rank * sizeof(float);
    if (dtype == IMPARO_DT_F32)
        launch(gla::decay_kernel<float>, grid, dim3(128), smem, stream, (const float*)low, (size_t)low_stride, (const float*)w2, bias, tau,
               out, n_tok, channels, rank);
    else if (dtype == IMPARO_DT_BF16)
        launch(gla::decay_kernel<__nv_bfloat16>, grid, dim3(128), smem, stream, (const __nv_bfloat16*)low, (size_t)low_stride,
               (const __nv_bfloat16*)w2, bias, tau, out, n_tok, channels, rank);
    else return -1;
    IMPARO_CHECK_LAUNCH();
    return 0;
}

// proj: rows of `stride` elements with q and k (heads * dim each) and v (heads * vdim) at the given columns; g float32
// [n_tok, heads * dim], the log decays; state float32 [n_slots, heads, dim, vdim]; out float32 [n_tok, heads * vdim].
extern "C" int imparo_gla_recurrent(const void* proj, long long stride, int dtype, int q_off, int k_off, int v_off, const float* g,
                                    float q_scale, float* state, const int* item_row_start, const int* item_slot, int n_slots,
                                    int n_items, float* out, int heads, int dim, int vdim, int* status, cudaStream_t stream) {
    if (n_items <= 0) return 0;
    if (heads < 1 || heads > 65535 || dim < 1 || dim > 256 || vdim < 1) return -2;
#define IMPARO_GL(T_) do { \
        gla::Cols<T_> c{(const T_*)proj, (size_t)stride, q_off, k_off, v_off, g, q_scale}; \
        if (dim <= 32) return gla::launch_recurrent<T_, 32>(c, state, item_row_start, item_slot, n_slots, n_items, out, heads, dim, vdim, status, stream); \
        if (dim <= 64) return gla::launch_recurrent<T_, 64>(c, state, item_row_start, item_slot, n_slots, n_items, out, heads, dim, vdim, status, stream); \
        if (dim <= 128) return gla::launch_recurrent<T_, 128>(c, state, item_row_start, item_slot, n_slots, n_items, out, heads, dim, vdim, status, stream); \
        return gla::launch_recurrent<T_, 256>(c, state, item_row_start, item_slot, n_slots, n_items, out, heads, dim, vdim, status, stream); } while (0)
    if (dtype == IMPARO_DT_F32) IMPARO_GL(float);
    if (dtype == IMPARO_DT_BF16) IMPARO_GL(__nv_bfloat16);
#undef IMPARO_GL
    return -1;
}

// Every request brings ONE row.  The columns of proj as above, the gate's (heads * vdim) at g_off, the decay's inner rows (rank) at
// l_off; w2 [heads * dim, rank] in proj's dtype, bias float32 [heads * dim]; w_norm float32 [vdim]; out [n_tok, heads * vdim] in
// proj's dtype = rms(o) * w_norm * silu(gate) per head.  vdim <= 512 (dim <= 64), 256 (<= 128) or 128; else -8.
extern "C" int imparo_gla_step(const void* proj, long long stride, int dtype, int q_off, int k_off, int v_off, int g_off, int l_off,
                               const void* w2, const float* bias, float tau, int rank, const float* w_norm, float eps, float q_scale,
                               float* state, const int* item_row_start, const int* item_slot, int n_slots, int n_items, void* out,
                               int heads, int dim, int vdim, int* status, cudaStream_t stream) {
    if (n_items <= 0) return 0;
    if (heads < 1 || heads > 65535 || dim < 1 || dim > 256 || vdim < 1 || rank < 1 || !(tau > 0.f)) return -2;
    const int wcols = dim > 128 ? 8 : (dim > 64 ? 16 : 32), warps = (vdim + wcols - 1) / wcols;
    if (warps > 16) return -8;
    const dim3 grid(n_items, heads), block(32 * warps);
#define IMPARO_GS(T_, D_, S_) launch(gla::step_kernel<T_, D_, S_>, grid, block, 0, stream, \
        gla::Cols<T_>{(const T_*)proj, (size_t)stride, q_off, k_off, v_off, nullptr, q_scale}, l_off, (const T_*)w2, bias, tau, rank, g_off, \
        w_norm, eps, state, item_row_start, item_slot, n_slots, (T_*)out, heads, dim, vdim, status)
#define IMPARO_GSD(T_) do { if (dim <= 32) IMPARO_GS(T_, 32, 1); else if (dim <= 64) IMPARO_GS(T_, 64, 1); \
        else if (dim <= 128) IMPARO_GS(T_, 128, 2); else IMPARO_GS(T_, 256, 4); } while (0)
    if (dtype == IMPARO_DT_F32) IMPARO_GSD(float);
    else if (dtype == IMPARO_DT_BF16) IMPARO_GSD(__nv_bfloat16);
    else return -1;
#undef IMPARO_GSD
#undef IMPARO_GS
    IMPARO_CHECK_LAUNCH();
    return 0;
}

// bfloat16 batches with long portions.  g float32 [n_tok, heads * dim]: the log decays, read; or, with w2 not null, made from the
// inner columns at l_off (rank <= 32) as imparo_gla_decay makes them and written.  dim and vdim multiples of 16, dim <= 128, 16-byte aligned columns; else -8.  chunk_state
// float32 [chunks, heads, dim, vdim] and chunk_decay [chunks, heads, dim] scratch, chunks = n_tok / 64 + n_items (an upper bound).
// vdim <= 128: y receives the normed, weighted, gated outputs (bfloat16 [n_tok, heads * vdim]); else o (float32) the plain ones.
extern "C" int imparo_gla_chunked(const void* proj, long long stride, int q_off, int k_off, int v_off, int g_off, int l_off, float* g,
                                  const void* w2, const float* bias, float tau, int rank, float q_scale, const float* w_norm, float eps, float* slots, const int* item_row_start,
                                  const int* item_slot, int n_slots, int n_items, int n_tok, float* chunk_state, float* chunk_decay,
                                  float* o, void* y, int heads, int dim, int vdim, int* status, cudaStream_t stream) {
    if (n_items <= 0 || n_tok <= 0) return 0;
    if (heads < 1 || heads > 65535 || n_items > 65535) return -2;
    if (dim < 16 || dim > 128 || dim % 16 || vdim < 16 || vdim % 16) return -8;
    if (stride % 8 || v_off % 8 || q_off % 2 || k_off % 2 || g_off % 2 || ((uintptr_t)proj & 15) || ((uintptr_t)g & 7)) return -8;
    if (((uintptr_t)slots | (uintptr_t)chunk_state) & 15) return -8;
    if (w2 != nullptr && (rank < 1 || rank > gla::MAX_RANK || bias == nullptr || !(tau > 0.f))) return -8;
    if (w2 == nullptr) rank = 0;
    const bool norm = vdim <= gla::CCOLS;
    if (norm ? y == nullptr : o == nullptr) return -2;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(gla::chunk_local_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gla::local_smem(128, 128, gla::MAX_RANK));
        if (e == cudaSuccess) e = cudaFuncSetAttribute(gla::chunk_local_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gla::local_smem(128, 128, 0));
        if (e == cudaSuccess) e = cudaFuncSetAttribute(gla::chunk_out_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gla::out_smem(128, 128));
        if (e == cudaSuccess) e = cudaFuncSetAttribute(gla::chunk_out_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gla::out_smem(128, 128));
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    gla::Chunks a;
    a.proj = (const __nv_bfloat16*)proj; a.stride = (size_t)stride;
    a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.g_off = g_off; a.g = g;
    a.l_off = l_off; a.rank = rank; a.w2 = (const __nv_bfloat16*)w2; a.bias = bias; a.tau = tau; a.q_scale = q_scale;
    a.item_row_start = item_row_start; a.n_items = n_items; a.state = chunk_state; a.decay = chunk_decay;
    a.heads = heads; a.dim = dim; a.vdim = vdim;
    const int vcols = vdim < gla::CCOLS ? vdim : gla::CCOLS;
    const dim3 grid(n_tok / gla::C + n_items, heads, (vdim + gla::CCOLS - 1) / gla::CCOLS);
    if (w2 != nullptr) launch(gla::chunk_local_kernel<true>, grid, dim3(gla::CT), gla::local_smem(dim, vcols, rank), stream, a);
    else launch(gla::chunk_local_kernel<false>, grid, dim3(gla::CT), gla::local_smem(dim, vcols, 0), stream, a);
    IMPARO_CHECK_LAUNCH();
    launch(gla::chunk_scan_kernel, dim3(n_items, heads, (dim * vdim / 4 + 255) / 256), dim3(256), 0, stream, a, slots, item_slot, n_slots, status);
    IMPARO_CHECK_LAUNCH();
    if (norm) launch(gla::chunk_out_kernel<true>, grid, dim3(gla::CT), gla::out_smem(dim, vcols), stream, a, w_norm, eps, o, (__nv_bfloat16*)y);
    else launch(gla::chunk_out_kernel<false>, grid, dim3(gla::CT), gla::out_smem(dim, vcols), stream, a, w_norm, eps, o, (__nv_bfloat16*)y);
    IMPARO_CHECK_LAUNCH();
    return 0;
}
