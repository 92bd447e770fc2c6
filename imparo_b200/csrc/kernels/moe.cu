// A routed feed-forward (mixture of experts) over the rows of a step.
//
//  (1) moe_route: router logits z = W_r h in 32-bit (a warp per expert, four rows per block), then a warp per row picks the
//      `top` largest (by logit: the scores sigmoid(z) or softmax(z) are monotone in it; ties: the lower expert), optionally
//      renormalised to sum 1.  Leaves expert ids [rows, top] and weights [rows, top].  With a correction per expert the choice
//      (and the groups' verdict) goes by score + correction, the weights by the score alone; a logit column behind the experts'
//      may give each row one more number, sigmoid(z) (the factor of an expert that every row uses).
//  (2) moe_few_*: steps of few rows (up to 256 pairs a launch), where reading the experts' matrices is the work.  A block belongs
//      to one of the experts the launch's pairs name and a stretch of its features; it finds its pairs itself and reads its matrix
//      rows once for up to eight or sixteen of their rows: in bfloat16 straight from global memory into tensor-core fragments
//      (mma.sync, sixteen matrix rows per block, its warps splitting the row length), else with the rows in shared memory and
//      scalar arithmetic.  The up kernel leaves act(..) per pair, the down kernel the (weighted) output per pair, which moe_sum adds
//      in the order of the choices.
//  (3) moe_group_*: pairs sorted by expert (a counting sort whose order inside an expert is the row order, so the
//      result does not depend on what else is in the step), tiles of 32 pairs x 64 outputs per CTA: bfloat16 on
//      tensor cores (mma.sync through wmma fragments, 32-bit accumulation), 32-bit with FFMA.  The tile list is made
//      on the device from the counts; CTAs beyond it leave at once, so the launch depends on (rows, top, experts)
//      only.
//
// Expert e's matrices: w_gu[e] = [gate; up] ([2 ff, width]), w_down[e] ([width, ff]); or, without a gate (gated = 0), w_gu[e] = up
// ([ff, width]) and one activation on its own (plain_act's kinds).  The weight multiplies the expert's input (weight_input = 1)
// or its output (0).
//
// A shared expert without a gate, of any size, may run in the launches of (2) as one more expert that every row uses.  Its rows'
// factors and the residual stream come in where the pairs are summed (moe_sum_pairs / moe_tile_sum), which can add into the stream
// and leave the rounded copy that the next product reads.
#include "common.cuh"
#include <mma.h>

namespace imparo {

// A warp's dot product of a matrix row with a vector in shared memory (32-bit).  When the row is 16 bytes wide per
// lane and turn (VEC), lanes read 16 bytes at a time, four loads in flight; the order of additions is fixed either way.
template <typename T> struct Vec16 { static constexpr int N = 16 / (int)sizeof(T); };

template <typename T>
__device__ __forceinline__ float dot16(const uint4 raw, const float* __restrict__ x) {
    float a = 0.f;
    if constexpr (sizeof(T) == 2) {
        const __nv_bfloat162* v = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const float2 f = __bfloat1622float2(v[u]);
            a = fmaf(f.x, x[2 * u], a);
            a = fmaf(f.y, x[2 * u + 1], a);
        }
    } else {
        const float* v = reinterpret_cast<const float*>(&raw);
#pragma unroll
        for (int u = 0; u < 4; ++u) a = fmaf(v[u], x[u], a);
    }
    return a;
}

// ---- (1) router -------------------------------------------------------------------------------------------------
// Logits: a block takes up to four rows (a router row read once serves them all) and eight experts, a warp each; grid
// (row blocks, ceil(experts / 8)).  A dot product always adds in the same order, whatever else the launch holds.
template <typename T>
__global__ void __launch_bounds__(256)
moe_logits_kernel(const T* __restrict__ h, const float* __restrict__ w_r, int n_rows, int width, int experts, int rows_per_block,
                  float* __restrict__ logits) {
    extern __shared__ __align__(16) float route_smem[];  // [rows][width] the rows in 32-bit
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r0 = blockIdx.x * rows_per_block;
    const int R = min(rows_per_block, n_rows - r0);
    float* rows = route_smem;
    for (int i = threadIdx.x; i < R * width; i += blockDim.x) rows[i] = to_f32(h[(size_t)r0 * width + i]);
    __syncthreads();
    const int e = blockIdx.y * 8 + warp;
    if (e >= experts) return;
    const float* wr = w_r + (size_t)e * width;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (width % 4 == 0) {
        const float4* w4 = reinterpret_cast<const float4*>(wr);
        const int n4 = width / 4;
        int i = lane;
        for (; i + 96 < n4; i += 128) {                      // four loads in flight
            float4 u[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) u[k] = w4[i + 32 * k];
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                if (r < R) {
                    const float* x = rows + (size_t)r * width + 4 * i;
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        acc[r] += u[k].x * x[128 * k] + u[k].y * x[128 * k + 1] + u[k].z * x[128 * k + 2] + u[k].w * x[128 * k + 3];
                }
            }
        }
        for (; i < n4; i += 32) {
            const float4 u = w4[i];
#pragma unroll
            for (int r = 0; r < 4; ++r)
                if (r < R) {
                    const float* x = rows + (size_t)r * width + 4 * i;
                    acc[r] += u.x * x[0] + u.y * x[1] + u.z * x[2] + u.w * x[3];
                }
        }
    } else {
        for (int i = lane; i < width; i += 32) {
            const float u = wr[i];
#pragma unroll
            for (int r = 0; r < 4; ++r)
                if (r < R) acc[r] += u * rows[(size_t)r * width + i];
        }
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const float v = warp_sum(acc[r]);
        if (lane == 0 && r < R) logits[(size_t)(r0 + r) * experts + e] = v;
    }
}

// The choice: a warp per row, four rows per block
// logits: [n_rows, parts * experts]; a logit is the sum of its `parts` entries, experts apart, added in order (parts > 1:
// the router matrix was cut into bfloat16 pieces whose sum is the 32-bit matrix to its last bit, see imparo_moe_pick)
// columns >= experts: the logits' columns per part (those beyond the experts' are not candidates); correction: float32
// [experts] or null; group_pair: a group's score is the sum of its two largest (else its largest); extra_out: float32 [n_rows]
// or null, sigmoid of column `experts`.
__global__ void __launch_bounds__(128)
moe_pick_kernel(const float* __restrict__ logits, int n_rows, int experts, int columns, int parts, int top, int softmax_scores,
                int renormalise, int groups, int keep, int group_pair, const float* __restrict__ correction, float renorm_eps,
                float weight_scale, int out_stride, int* __restrict__ ids, float* __restrict__ wts, float* __restrict__ extra_out) {
    extern __shared__ __align__(16) float pick_smem[];   // [4][experts] scores, then [4][groups] scores of the groups
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r = blockIdx.x * 4 + warp;
    if (r >= n_rows) return;
    float* s = pick_smem + (size_t)warp * experts;
    auto logit = [&](int e) {
        const float* l = logits + (size_t)r * parts * columns + e;
        float v = l[0];
        for (int k = 1; k < parts; ++k) v += l[(size_t)k * columns];
        return v;
    };
    for (int e = lane; e < experts; e += 32) {
        const float v = logit(e);
        s[e] = correction ? 1.0f / (1.0f + expf(-v)) + correction[e] : v;
    }
    if (extra_out && lane == 0) extra_out[r] = 1.0f / (1.0f + expf(-logit(experts)));
    __syncwarp();
    // Without a correction the choice goes by the logits: scores are monotone in them, and a sigmoid that has reached 1 in
    // 32-bit would tie.
    float m = -INFINITY, l = 1.f;
    if (softmax_scores) {
        for (int e = lane; e < experts; e += 32) m = fmaxf(m, s[e]);
        m = warp_max(m);
        l = 0.f;
        for (int e = lane; e < experts; e += 32) l += expf(s[e] - m);
        l = warp_sum(l);
    }
    // Experts in `groups` equal groups of neighbours: a group's score is its largest (or the sum of its two largest), and only
    // the `keep` best groups' experts stay candidates (ties: the lower group).  The others leave the candidates; the softmax
    // above counted them.
    if (groups > 1 && keep < groups) {
        const int per = experts / groups;
        // every group's score first (a lane per group), then a lane per group counts the groups that beat its own: a group
        // is kept when fewer than `keep` do.  All verdicts are in before any score is masked.
        float* gmax = pick_smem + (size_t)4 * experts + (size_t)warp * groups;
        for (int g = lane; g < groups; g += 32) {
            float mx = -INFINITY, second = -INFINITY;
            for (int e = g * per; e < (g + 1) * per; ++e) {
                const float v = s[e];
                second = fmaxf(second, fminf(mx, v));
                mx = fmaxf(mx, v);
            }
            gmax[g] = group_pair && per > 1 ? mx + second : mx;
        }
        __syncwarp();
        for (int g = lane; g < groups; g += 32) {
            const float mine = gmax[g];
            int beaten = 0;
            for (int o = 0; o < groups; ++o) {
                const float other = gmax[o];
                if (other > mine || (other == mine && o < g)) ++beaten;
            }
            if (beaten >= keep)
                for (int e = g * per; e < (g + 1) * per; ++e) s[e] = -INFINITY;
        }
        __syncwarp();
    }
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int arg = 0x7fffffff;
        for (int e = lane; e < experts; e += 32) {
            const float v = s[e];
            if (v > best) { best = v; arg = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
            if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
        }
        const float score = softmax_scores ? expf(best - m) / l : 1.0f / (1.0f + expf(-(correction ? logit(arg) : best)));
        if (lane == 0) {
            ids[(size_t)r * out_stride + k] = arg;
            wts[(size_t)r * out_stride + k] = score;
            s[arg] = -INFINITY;
        }
        total += score;
        __syncwarp();
    }
    if (renormalise && lane < top) wts[(size_t)r * out_stride + lane] = wts[(size_t)r * out_stride + lane] / (total + renorm_eps) * weight_scale;
    else if (weight_scale != 1.0f && lane < top) wts[(size_t)r * out_stride + lane] *= weight_scale;
    // choices beyond `top` (out_stride > top) are experts every row uses with weight 1: numbers experts, experts + 1, ...
    for (int k = top + lane; k < out_stride; k += 32) {
        ids[(size_t)r * out_stride + k] = experts + (k - top);
        wts[(size_t)r * out_stride + k] = 1.0f;
    }
}

// ---- (2) few rows ---------------------------------------------------------------------------------------------------
constexpr int FEW_ROWS = 8, FEW_PAIRS = 256;          // rows a block works on at once; pairs a launch may have

// acc[j][r] = w[j] . x row r for four matrix rows (null: left out) and the block's rows; xs: [rows][n] in shared memory.  A lane
// takes every 32nd 16 bytes of a row, two of them in flight; the sums end with a fixed tree over the warp.
template <typename T>
__device__ __forceinline__ void warp_dot_rows(const T* const (&w)[4], const T* xs, int rows, int n, bool vec, int lane,
                                              float (&acc)[4][FEW_ROWS]) {
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int r = 0; r < FEW_ROWS; ++r) acc[j][r] = 0.f;
    if (vec) {
        constexpr int PER = Vec16<T>::N;
        const int n4 = n / PER;
        auto part = [&](const uint4 (&wv)[4], int i) {
#pragma unroll
            for (int r = 0; r < FEW_ROWS; ++r) {
                if (r >= rows) break;
                const uint4 xv = reinterpret_cast<const uint4*>(xs + (size_t)r * n)[i];
                float xf[PER];
#pragma unroll
                for (int u = 0; u < PER; ++u) xf[u] = to_f32(reinterpret_cast<const T*>(&xv)[u]);
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[j][r] += dot16<T>(wv[j], xf);
            }
        };
        auto load = [&](uint4 (&wv)[4], int i) {
#pragma unroll
            for (int j = 0; j < 4; ++j) wv[j] = w[j] ? __ldg(reinterpret_cast<const uint4*>(w[j]) + i) : make_uint4(0u, 0u, 0u, 0u);
        };
        int i = lane;
        for (; i + 32 < n4; i += 64) {
            uint4 a[4], b[4];
            load(a, i);
            load(b, i + 32);
            part(a, i);
            part(b, i + 32);
        }
        if (i < n4) {
            uint4 a[4];
            load(a, i);
            part(a, i);
        }
    } else {
        for (int i = lane; i < n; i += 32)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (w[j] == nullptr) continue;
                const float wv = to_f32(w[j][i]);
#pragma unroll
                for (int r = 0; r < FEW_ROWS; ++r) if (r < rows) acc[j][r] += wv * to_f32(xs[(size_t)r * n + i]);
            }
    }
#pragma unroll
    for (int r = 0; r < FEW_ROWS; ++r) {
        if (r >= rows) break;
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[j][r] = warp_sum(acc[j][r]);
    }
}

// What an expert-by-expert launch does besides the routed experts (w null: nothing): an ungated expert with `n_feat` matrix rows
// of `n` entries that every row uses; in: [n_rows, n], out: [n_rows, n_feat].
struct SharedRows {
    const void* w;
    const void* in;
    void* out;
    int n_feat, n;
};

// The launch's pairs as a block sees them: the k-th of the experts they name (-1: there are fewer), its pairs (in order) in list,
// and how many.  Up to 32 pairs every warp finds the answer by itself; with more the block first marks the experts in a bit set.
// (All warps write the same list.)  Every thread of the block calls it.
constexpr int FEW_EXPERTS = 2048;
__device__ __forceinline__ int few_pairs_of(const int* __restrict__ ids, int n_pairs, int experts, int k, int* list, int& count) {
    const int lane = threadIdx.x & 31;
    const unsigned below = (1u << lane) - 1u;
    if (n_pairs <= 32) {
        int id = lane < n_pairs ? ids[lane] : -1;
        if (id >= experts) id = -1;
        const unsigned same = __match_any_sync(0xffffffffu, id);
        const bool first = id >= 0 && (same & below) == 0;
        const unsigned firsts = __ballot_sync(0xffffffffu, first);
        const unsigned hit = __ballot_sync(0xffffffffu, first && __popc(firsts & below) == k);
        if (hit == 0) return -1;
        const int src = __ffs(hit) - 1;
        const int e = __shfl_sync(0xffffffffu, id, src);
        const unsigned members = __shfl_sync(0xffffffffu, same, src);
        if ((members >> lane) & 1u) list[__popc(members & below)] = lane;
        __syncwarp();
        count = __popc(members);
        return e;
    }
    __shared__ unsigned named[FEW_EXPERTS / 32];
    for (int i = threadIdx.x; i < FEW_EXPERTS / 32; i += blockDim.x) named[i] = 0u;
    __syncthreads();
    for (int p = threadIdx.x; p < n_pairs; p += blockDim.x) {
        const int id = ids[p];
        if (id >= 0 && id < experts) atomicOr(&named[id >> 5], 1u << (id & 31));
    }
    __syncthreads();
    // a lane looks at two words; a running count over the lanes finds the word with the k-th expert
    unsigned w0 = named[2 * lane], w1 = named[2 * lane + 1];
    const int mine = __popc(w0) + __popc(w1);
    int upto = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, upto, o);
        if (lane >= o) upto += v;
    }
    int e = -1;
    if (k < upto && k >= upto - mine) {
        int left = k - (upto - mine), base = 64 * lane;
        unsigned word = w0;
        if (left >= __popc(w0)) { left -= __popc(w0); word = w1; base += 32; }
        for (; left > 0; --left) word &= word - 1;
        e = base + __ffs(word) - 1;
    }
    const unsigned hit = __ballot_sync(0xffffffffu, e >= 0);
    if (hit == 0) return -1;
    e = __shfl_sync(0xffffffffu, e, __ffs(hit) - 1);
    int n = 0;
    for (int p0 = 0; p0 < n_pairs; p0 += 32) {
        const bool member = p0 + lane < n_pairs && ids[p0 + lane] == e;
        const unsigned m = __ballot_sync(0xffffffffu, member);
        if (member) list[n + __popc(m & below)] = p0 + lane;
        n += __popc(m);
    }
    __syncwarp();
    count = n;
    return e;
}

// Blocks: grid (shared row tiles + experts at most, feature stretches), 256 threads; a warp works on four matrix rows: four
// features, or the gate and up rows of two (gated).
//   UP:   in = h [n_rows, n], matrices [features (2x with gated), n], out = mid [pairs, features] in T: act(..)
//   down: in = mid [pairs, n], matrices [features, n], out = pair_out float32 [pairs, features], times the weight unless weight_input
template <typename T, bool UP>
__global__ void __launch_bounds__(256, 2)
moe_few_kernel(const T* __restrict__ in, const T* __restrict__ w, const int* __restrict__ ids, const float* __restrict__ wts, int n_rows,
               int n, int n_feat, int top, int experts, int weight_input, int gated, int act, float limit, void* __restrict__ out,
               SharedRows sh) {
    extern __shared__ __align__(16) uint8_t few_smem[];
    __shared__ int list[FEW_PAIRS];
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    T* xs = reinterpret_cast<T*>(few_smem);
    // the shared expert's blocks come first: they have the most to do
    const int shared_tiles = sh.w ? (n_rows + FEW_ROWS - 1) / FEW_ROWS : 0;
    const bool shared = (int)blockIdx.x < shared_tiles;
    if (shared) { n = sh.n; n_feat = sh.n_feat; gated = 0; }
    const int per_warp = gated ? 2 : 4, f_block = blockIdx.y * 8 * per_warp;
    if (f_block >= n_feat) return;
    int e = 0, count = n_rows;
    if (!shared) {
        e = few_pairs_of(ids, n_rows * top, experts, blockIdx.x - shared_tiles, list, count);
        if (e < 0) return;
    }
    const T* src = shared ? (const T*)sh.in : in;
    const T* mat = shared ? (const T*)sh.w : w + (size_t)e * (gated ? 2 : 1) * n_feat * n;
    const bool vec = n % Vec16<T>::N == 0 && (((uintptr_t)mat | (uintptr_t)src) & 15) == 0;
    const int f0 = f_block + warp * per_warp;
    const T* rowp[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int f = gated ? f0 + (j >> 1) : f0 + j;
        rowp[j] = f < n_feat ? mat + (size_t)((gated && (j & 1)) ? n_feat + f : f) * n : nullptr;
    }
    const int lo = shared ? blockIdx.x * FEW_ROWS : 0, hi = shared ? min(n_rows, lo + FEW_ROWS) : count;
    for (int r0 = lo; r0 < hi; r0 += FEW_ROWS) {
        const int rows = min(FEW_ROWS, hi - r0);
        __syncthreads();                                   // the rows before have been read
        for (int r = 0; r < rows; ++r) {
            const int item = shared ? r0 + r : list[r0 + r];
            const T* xr = src + (size_t)(UP && !shared ? item / top : item) * n;
            const float wt = UP && weight_input && !shared ? wts[item] : 1.0f;
            if (vec) {
                for (int i = threadIdx.x; i < n / Vec16<T>::N; i += 256) {
                    uint4 raw = reinterpret_cast<const uint4*>(xr)[i];
                    if (UP && weight_input && !shared) {
                        T* v = reinterpret_cast<T*>(&raw);
#pragma unroll
                        for (int u = 0; u < Vec16<T>::N; ++u) v[u] = from_f32<T>(wt * to_f32(v[u]));
                    }
                    reinterpret_cast<uint4*>(xs + (size_t)r * n)[i] = raw;
                }
            } else {
                for (int i = threadIdx.x; i < n; i += 256) xs[(size_t)r * n + i] = from_f32<T>(wt * to_f32(xr[i]));
            }
        }
        __syncthreads();
        if (f0 >= n_feat) continue;
        float acc[4][FEW_ROWS];
        warp_dot_rows<T>(rowp, xs, rows, n, vec, lane, acc);
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int r = 0; r < FEW_ROWS; ++r) {
                if (lane != j * FEW_ROWS + r || r >= rows) continue;
                const int item = shared ? r0 + r : list[r0 + r];
                if (gated) {
                    const int f = f0 + (j >> 1);
                    if ((j & 1) == 0 && f < n_feat)
                        reinterpret_cast<T*>(out)[(size_t)item * n_feat + f] = from_f32<T>(gated_act(act, limit, acc[j][r], acc[(j + 1) & 3][r]));
                } else if (f0 + j < n_feat) {
                    const size_t at = (size_t)item * n_feat + f0 + j;
                    if (UP) reinterpret_cast<T*>(shared ? sh.out : out)[at] = from_f32<T>(plain_act(act, acc[j][r]));
                    else if (shared) reinterpret_cast<float*>(sh.out)[at] = acc[j][r];
                    else reinterpret_cast<float*>(out)[at] = (weight_input ? 1.0f : wts[item]) * acc[j][r];
                }
            }
    }
}

// ---- few rows in bfloat16 on tensor cores ----------------------------------------------------------------------------
constexpr int MM_WARPS = 8, MM_ROUND = 4;              // warps of a block; 32-entry stretches a warp has in flight

__device__ __forceinline__ uint4 ld_stream(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ void mma_16x8x16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// As moe_few_kernel, with 16 matrix rows per block (gated: the gate and up rows of eight features) and NB tiles of eight rows at
// once.  A warp takes every MM_WARPS-th round of 32-entry stretches of the row length.  In a stretch lane (g, t) of the warp holds
// entries 8 t .. 8 t + 7 of matrix rows g and g + 8 and of row g of the operand, 16 bytes each: a dot product does not mind in which
// order its terms are taken, so the four entries that an mma calls k = 2t, 2t + 1, 2t + 8, 2t + 9 are the lane's own neighbours, in
// both operands.  The warps' partial sums are added in warp order.  n a multiple of 8, 16-byte aligned pointers.
template <bool UP, int NB>
__global__ void __launch_bounds__(MM_WARPS * 32, NB == 1 ? 4 : 2)
moe_few_mma_kernel(const __nv_bfloat16* __restrict__ in, const __nv_bfloat16* __restrict__ w, const int* __restrict__ ids,
                   const float* __restrict__ wts, int n_rows, int n, int n_feat, int top, int experts, int weight_input, int gated, int act,
                   float limit, void* __restrict__ out, SharedRows sh) {
    using T = __nv_bfloat16;
    __shared__ int list[FEW_PAIRS];
    __shared__ __align__(16) float part[MM_WARPS][NB][128];
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int shared_tiles = sh.w ? (n_rows + 8 * NB - 1) / (8 * NB) : 0;
    const bool shared = (int)blockIdx.x < shared_tiles;
    if (shared) { n = sh.n; n_feat = sh.n_feat; gated = 0; }
    const int f0 = blockIdx.y * (gated ? 8 : 16);
    if (f0 >= n_feat) return;
    int e = 0, count = n_rows;
    if (!shared) {
        e = few_pairs_of(ids, n_rows * top, experts, blockIdx.x - shared_tiles, list, count);
        if (e < 0) return;
    }
    const T* src = shared ? (const T*)sh.in : in;
    const T* mat = shared ? (const T*)sh.w : w + (size_t)e * (gated ? 2 : 1) * n_feat * n;
    const int fa = f0 + g, fb = gated ? f0 + g : f0 + g + 8;
    const T* ra = fa < n_feat ? mat + (size_t)fa * n + 8 * t : nullptr;
    const T* rb = fb < n_feat ? mat + (size_t)(gated ? n_feat + fb : fb) * n + 8 * t : nullptr;
    const int lo = shared ? blockIdx.x * 8 * NB : 0, hi = shared ? min(n_rows, lo + 8 * NB) : count;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    for (int r0 = lo; r0 < hi; r0 += 8 * NB) {
        const T* xr[NB];
        float xw[NB];
        float acc[NB][4];
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            const int r = r0 + 8 * b + g;
            xr[b] = nullptr;
            xw[b] = 1.f;
            acc[b][0] = acc[b][1] = acc[b][2] = acc[b][3] = 0.f;
            if (r < hi) {
                const int item = shared ? r : list[r];
                xr[b] = src + (size_t)(UP && !shared ? item / top : item) * n + 8 * t;
                if (UP && weight_input && !shared) xw[b] = wts[item];
            }
        }
        for (int k0 = warp * MM_ROUND * 32; k0 < n; k0 += MM_WARPS * MM_ROUND * 32) {
            uint4 a[MM_ROUND], c[MM_ROUND], x[MM_ROUND][NB];             // all loads of a round are in flight at once
#pragma unroll
            for (int u = 0; u < MM_ROUND; ++u) {
                const int k = k0 + 32 * u;
                const bool live = k + 8 * t < n;
                a[u] = live && ra ? ld_stream(ra + k) : zero;
                c[u] = live && rb ? ld_stream(rb + k) : zero;
            }
#pragma unroll
            for (int u = 0; u < MM_ROUND; ++u)
#pragma unroll
                for (int b = 0; b < NB; ++b) {
                    const int k = k0 + 32 * u;
                    x[u][b] = k + 8 * t < n && xr[b] ? *reinterpret_cast<const uint4*>(xr[b] + k) : zero;
                }
#pragma unroll
            for (int u = 0; u < MM_ROUND; ++u) {
                if (k0 + 32 * u >= n) break;
#pragma unroll
                for (int b = 0; b < NB; ++b) {
                    uint4 xv = x[u][b];
                    if (UP && weight_input && !shared) {
                        __nv_bfloat162* v = reinterpret_cast<__nv_bfloat162*>(&xv);
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            const float2 f = __bfloat1622float2(v[i]);
                            v[i] = __floats2bfloat162_rn(xw[b] * f.x, xw[b] * f.y);
                        }
                    }
                    mma_16x8x16(acc[b], a[u].x, c[u].x, a[u].y, c[u].y, xv.x, xv.y);
                    mma_16x8x16(acc[b], a[u].z, c[u].z, a[u].w, c[u].w, xv.z, xv.w);
                }
            }
        }
        __syncthreads();                                   // the sums before have been read
#pragma unroll
        for (int b = 0; b < NB; ++b)
            *reinterpret_cast<float4*>(&part[warp][b][lane * 4]) = make_float4(acc[b][0], acc[b][1], acc[b][2], acc[b][3]);
        __syncthreads();
        // thread = (lane's place, which of its four sums): 0, 1: matrix row g, rows 2t and 2t + 1; 2, 3: matrix row g + 8
        const int pl = (threadIdx.x & 127) >> 2, pc = threadIdx.x & 3, pg = pl >> 2, pt = pl & 3;
#pragma unroll
        for (int b = threadIdx.x >> 7; b < NB; b += 2) {
            const int r = r0 + 8 * b + 2 * pt + (pc & 1);
            if (r >= hi) continue;
            const int item = shared ? r : list[r];
            float v = 0.f, v2 = 0.f;
#pragma unroll
            for (int k = 0; k < MM_WARPS; ++k) v += part[k][b][pl * 4 + pc];
            if (gated) {
                if (pc >= 2) continue;
#pragma unroll
                for (int k = 0; k < MM_WARPS; ++k) v2 += part[k][b][pl * 4 + pc + 2];
                if (f0 + pg < n_feat) reinterpret_cast<T*>(out)[(size_t)item * n_feat + f0 + pg] = from_f32<T>(gated_act_bf16(act, limit, v, v2));
                continue;
            }
            const int f = f0 + pg + (pc >> 1) * 8;
            if (f >= n_feat) continue;
            const size_t at = (size_t)item * n_feat + f;
            if (UP) reinterpret_cast<T*>(shared ? sh.out : out)[at] = from_f32<T>(plain_act_bf16(act, v));
            else if (shared) reinterpret_cast<float*>(sh.out)[at] = v;
            else reinterpret_cast<float*>(out)[at] = (weight_input ? 1.0f : wts[item]) * v;
        }
    }
}

// ---- (3) grouped by expert ----------------------------------------------------------------------------------------
constexpr int GM = 32, GN = 64, GK = 32;          // tile: pairs x outputs, K step

// One block: counts per expert, offsets, the sorted pair list (stable: by expert, then by pair index) and the tile list.
// plan: [0] number of tiles; tile_expert[t], tile_first[t] (index into sorted), tile_rows[t]
__global__ void __launch_bounds__(1024)
moe_group_plan_kernel(const int* __restrict__ ids, int n_pairs, int experts, int* __restrict__ sorted,
                      int* __restrict__ expert_start, int* __restrict__ plan, int max_tiles) {
    extern __shared__ int plan_smem[];               // experts + 1 offsets
    pdl_trigger();
    pdl_wait();
    int* start = plan_smem;
    const int tid = threadIdx.x;
    // thread e counts its expert's pairs and then writes them in pair order: the order inside an expert is by row
    for (int e = tid; e <= experts; e += blockDim.x) start[e] = 0;
    __syncthreads();
    for (int e = tid; e < experts; e += blockDim.x) {
        int c = 0;
        for (int i = 0; i < n_pairs; ++i) c += ids[i] == e;
        start[e + 1] = c;
    }
    __syncthreads();
    if (tid == 0) {
        int tiles = 0;
        for (int e = 0; e < experts; ++e) {
            const int c = start[e + 1];
            start[e + 1] = start[e] + c;
            for (int lo = 0; lo < c && tiles < max_tiles; lo += GM) {
                plan[1 + 3 * tiles] = e;
                plan[2 + 3 * tiles] = start[e] + lo;
                plan[3 + 3 * tiles] = min(GM, c - lo);
                ++tiles;
            }
        }
        plan[0] = tiles;
    }
    __syncthreads();
    for (int e = tid; e < experts; e += blockDim.x) {
        int at = start[e];
        expert_start[e] = at;
        for (int i = 0; i < n_pairs; ++i)
            if (ids[i] == e) sorted[at++] = i;
    }
    if (tid == 0) expert_start[experts] = start[experts];
}

// A[m, k]: row `pair_of[m]` of the operand (times its weight when asked), B[n, k]: the expert's matrix rows.
// bfloat16: wmma 16x16x16, 8 warps as 2 (m) x 4 (n); float32: each thread a 2 x 4 patch with FFMA.
template <typename T> struct GroupTile;

template <> struct __align__(32) GroupTile<__nv_bfloat16> {
    using T = __nv_bfloat16;
    static constexpr int LDS = GK + 8;
    T a[GM][LDS];
    T b[GN][LDS];
    float c[GM][GN + 4];
};
template <> struct __align__(32) GroupTile<float> {
    static constexpr int LDS = GK + 1;
    float a[GM][LDS];
    float b[GN][LDS];
    float c[GM][GN + 4];
};

// acc tile = A (GM x K) * B^T (GN x K); result left in sm.c
template <typename T, typename LoadA>
__device__ __forceinline__ void group_tile_product(GroupTile<T>& sm, LoadA load_a, const T* __restrict__ bmat, int n0, int n_rows_b,
                                                   int K, int rows) {
    const int tid = threadIdx.x;
    if constexpr (sizeof(T) == 2) {
        using namespace nvcuda;
        const int warp = tid >> 5, wm = warp >> 2, wn = warp & 3;
        wmma::fragment<wmma::accumulator, 16, 16, 16, float> acc;
        wmma::fill_fragment(acc, 0.f);
        for (int k0 = 0; k0 < K; k0 += GK) {
            __syncthreads();
            for (int i = tid; i < GM * GK; i += 256) {
                const int m = i / GK, k = i % GK;
                sm.a[m][k] = (m < rows && k0 + k < K) ? load_a(m, k0 + k) : from_f32<T>(0.f);
            }
            for (int i = tid; i < GN * GK; i += 256) {
                const int n = i / GK, k = i % GK;
                sm.b[n][k] = (n0 + n < n_rows_b && k0 + k < K) ? bmat[(size_t)(n0 + n) * K + k0 + k] : from_f32<T>(0.f);
            }
            __syncthreads();
#pragma unroll
            for (int kk = 0; kk < GK; kk += 16) {
                wmma::fragment<wmma::matrix_a, 16, 16, 16, __nv_bfloat16, wmma::row_major> fa;
                wmma::fragment<wmma::matrix_b, 16, 16, 16, __nv_bfloat16, wmma::col_major> fb;
                wmma::load_matrix_sync(fa, &sm.a[wm * 16][kk], GroupTile<T>::LDS);
                wmma::load_matrix_sync(fb, &sm.b[wn * 16][kk], GroupTile<T>::LDS);
                wmma::mma_sync(acc, fa, fb, acc);
            }
        }
        wmma::store_matrix_sync(&sm.c[wm * 16][wn * 16], acc, GN + 4, wmma::mem_row_major);
        __syncthreads();
    } else {
        const int tm = (tid >> 4) * 2, tn = (tid & 15) * 4;      // 16 x 16 threads, 2 x 4 each
        float acc[2][4] = {};
        for (int k0 = 0; k0 < K; k0 += GK) {
            __syncthreads();
            for (int i = tid; i < GM * GK; i += 256) {
                const int m = i / GK, k = i % GK;
                sm.a[m][k] = (m < rows && k0 + k < K) ? load_a(m, k0 + k) : 0.f;
            }
            for (int i = tid; i < GN * GK; i += 256) {
                const int n = i / GK, k = i % GK;
                sm.b[n][k] = (n0 + n < n_rows_b && k0 + k < K) ? bmat[(size_t)(n0 + n) * K + k0 + k] : 0.f;
            }
            __syncthreads();
            const int kn = min(GK, K - k0);
            for (int k = 0; k < kn; ++k) {
                float av[2], bv[4];
#pragma unroll
                for (int i = 0; i < 2; ++i) av[i] = sm.a[tm + i][k];
#pragma unroll
                for (int j = 0; j < 4; ++j) bv[j] = sm.b[tn + j][k];
#pragma unroll
                for (int i = 0; i < 2; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[i][j] += av[i] * bv[j];
            }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) sm.c[tm + i][tn + j] = acc[i][j];
        __syncthreads();
    }
}

// grid (max_tiles, ceil(ff / 64)): mid[pair, f] = silu(gate) * up for the tile's pairs; gate and up as two products
template <typename T>
__global__ void __launch_bounds__(256)
moe_group_up_kernel(const T* __restrict__ h, const T* __restrict__ w_gu, const int* __restrict__ sorted, const int* __restrict__ plan,
                    const float* __restrict__ wts, int width, int ff, int top, int weight_input, int gated, int act, float limit,
                    T* __restrict__ mid) {
    __shared__ GroupTile<T> sm;
    __shared__ int pair_of[GM];
    __shared__ float wt_of[GM];
    __shared__ float gate_c[GM][GN];
    pdl_trigger();
    pdl_wait();
    const int tile = blockIdx.x;
    if (tile >= plan[0]) return;
    const int e = plan[1 + 3 * tile], first = plan[2 + 3 * tile], rows = plan[3 + 3 * tile];
    if (threadIdx.x < GM) {
        const int p = threadIdx.x < rows ? sorted[first + threadIdx.x] : -1;
        pair_of[threadIdx.x] = p;
        wt_of[threadIdx.x] = (p >= 0 && weight_input) ? wts[p] : 1.0f;
    }
    __syncthreads();
    const int n0 = blockIdx.y * GN;
    auto load_a = [&](int m, int k) -> T {
        return from_f32<T>(wt_of[m] * to_f32(h[(size_t)(pair_of[m] / top) * width + k]));
    };
    const T* base = w_gu + (size_t)e * (gated ? 2 : 1) * ff * width;
    group_tile_product<T>(sm, load_a, base, n0, ff, width, rows);
    if (!gated) {
        for (int i = threadIdx.x; i < GM * GN; i += 256) {
            const int m = i / GN, n = i % GN;
            if (m < rows && n0 + n < ff) mid[(size_t)pair_of[m] * ff + n0 + n] = from_f32<T>(plain_act(act, sm.c[m][n]));
        }
        return;
    }
    for (int i = threadIdx.x; i < GM * GN; i += 256) gate_c[i / GN][i % GN] = sm.c[i / GN][i % GN];
    group_tile_product<T>(sm, load_a, base + (size_t)ff * width, n0, ff, width, rows);
    for (int i = threadIdx.x; i < GM * GN; i += 256) {
        const int m = i / GN, n = i % GN;
        if (m < rows && n0 + n < ff) mid[(size_t)pair_of[m] * ff + n0 + n] = from_f32<T>(gated_act(act, limit, gate_c[m][n], sm.c[m][n]));
    }
}

// grid (max_tiles, ceil(width / 64)): pair_out[pair, o] = down row o . mid[pair]  (times the weight when it is on the output)
template <typename T>
__global__ void __launch_bounds__(256)
moe_group_down_kernel(const T* __restrict__ mid, const T* __restrict__ w_down, const int* __restrict__ sorted,
                      const int* __restrict__ plan, const float* __restrict__ wts, int width, int ff, int weight_input,
                      float* __restrict__ pair_out) {
    __shared__ GroupTile<T> sm;
    __shared__ int pair_of[GM];
    pdl_trigger();
    pdl_wait();
    const int tile = blockIdx.x;
    if (tile >= plan[0]) return;
    const int e = plan[1 + 3 * tile], first = plan[2 + 3 * tile], rows = plan[3 + 3 * tile];
    if (threadIdx.x < GM) pair_of[threadIdx.x] = threadIdx.x < rows ? sorted[first + threadIdx.x] : -1;
    __syncthreads();
    const int n0 = blockIdx.y * GN;
    auto load_a = [&](int m, int k) -> T { return mid[(size_t)pair_of[m] * ff + k]; };
    group_tile_product<T>(sm, load_a, w_down + (size_t)e * width * ff, n0, width, ff, rows);
    for (int i = threadIdx.x; i < GM * GN; i += 256) {
        const int m = i / GN, n = i % GN;
        if (m < rows && n0 + n < width) {
            const float wt = weight_input ? 1.0f : wts[pair_of[m]];
            pair_out[(size_t)pair_of[m] * width + n0 + n] = wt * sm.c[m][n];
        }
    }
}

// What the sums below may do besides: add extra_w[r] * extra[r, :] (extra float32 [rows, width], extra_w float32 [rows]; null:
// nothing), add into what `out` holds (accumulate), and leave the result's rows rounded in `copy` (bfloat16 or null).
struct SumTail {
    const float* extra;
    const float* extra_w;
    int accumulate;
    __nv_bfloat16* copy;
};

// out[r, :] = sum over the row's choices, in order; VEC: four columns at a time (width a multiple of 4, 16-byte aligned)
template <bool VEC>
__global__ void __launch_bounds__(256)
moe_sum_pairs_kernel(const float* __restrict__ pair_out, int n_rows, int width, int top, float* __restrict__ out, SumTail tail) {
    pdl_trigger();
    pdl_wait();
    constexpr int N = VEC ? 4 : 1;
    const size_t total = (size_t)n_rows * width / N;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t r = i * N / width, c = i * N - r * width;
        float a[N];
#pragma unroll
        for (int u = 0; u < N; ++u) a[u] = 0.f;
        auto add = [&](const float* p, float f) {
            if constexpr (VEC) {
                const float4 v = *reinterpret_cast<const float4*>(p);
                a[0] += f * v.x; a[1] += f * v.y; a[2] += f * v.z; a[3] += f * v.w;
            } else {
                a[0] += f * *p;
            }
        };
        for (int k = 0; k < top; ++k) add(pair_out + (r * top + k) * width + c, 1.f);
        if (tail.extra) add(tail.extra + r * width + c, tail.extra_w[r]);
        if (tail.accumulate) add(out + r * width + c, 1.f);
        if constexpr (VEC) {
            *reinterpret_cast<float4*>(out + r * width + c) = make_float4(a[0], a[1], a[2], a[3]);
            if (tail.copy) {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(a[0], a[1]), hi = __floats2bfloat162_rn(a[2], a[3]);
                *reinterpret_cast<uint2*>(tail.copy + r * width + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo),
                                                                                  *reinterpret_cast<const uint32_t*>(&hi));
            }
        } else {
            out[r * width + c] = a[0];
            if (tail.copy) tail.copy[r * width + c] = __float2bfloat16(a[0]);
        }
    }
}

// ---- (4) sorted into tiles of 128 rows for the tensor-memory product (gemm_prefill.cu, grouped) --------------------------
// One block.  Every pair gets a row in a buffer in which each expert's rows start at a multiple of 128: slot_of_pair[p];
// tile_group[t] names the expert of row tile t, -1 beyond the last used tile.  Inside an expert the rows keep the pairs'
// order.  Shared memory: (32 + 2) * experts ints.
constexpr int TILE_ROWS = 128;

__global__ void __launch_bounds__(1024)
moe_tile_plan_kernel(const int* __restrict__ ids, int n_pairs, int experts, int* __restrict__ slot_of_pair,
                     int* __restrict__ tile_group, int max_tiles) {
    extern __shared__ int tp_smem[];
    int* counts = tp_smem;                               // [32][experts] pairs per warp's stretch, then those before the stretch
    int* total = tp_smem + 32 * experts;                 // [experts]
    int* start_row = total + experts;                    // [experts] first row of the expert's stretch
    __shared__ int used_tiles;
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    for (int i = tid; i < 32 * experts; i += blockDim.x) counts[i] = 0;
    __syncthreads();
    // every warp ranks the pairs of its own stretch, in order, without a word to the others
    const int per = ((n_pairs + 31) / 32 + 31) / 32 * 32, p0 = warp * per, p1 = min(n_pairs, p0 + per);
    int* mine = counts + warp * experts;
    for (int p = p0 + lane; p - lane < p1; p += 32) {
        int e = p < p1 ? ids[p] : -1;
        if (e >= experts) e = -1;
        const unsigned same = __match_any_sync(0xffffffffu, e);
        const int rank = __popc(same & ((1u << lane) - 1u));
        const int before = e >= 0 ? mine[e] : 0;
        __syncwarp();
        if (e >= 0 && rank == 0) mine[e] = before + __popc(same);
        __syncwarp();
        if (p < p1) slot_of_pair[p] = e >= 0 ? before + rank : -1;
    }
    __syncthreads();
    for (int x = tid; x < experts; x += blockDim.x) {
        int run = 0;
        for (int w = 0; w < 32; ++w) {
            const int c = counts[w * experts + x];
            counts[w * experts + x] = run;
            run += c;
        }
        total[x] = run;
    }
    __syncthreads();
    if (tid == 0) {
        int t = 0;
        for (int e = 0; e < experts; ++e) {
            start_row[e] = t * TILE_ROWS;
            t += (total[e] + TILE_ROWS - 1) / TILE_ROWS;
        }
        used_tiles = min(t, max_tiles);
    }
    __syncthreads();
    for (int e = tid; e < experts; e += blockDim.x) {
        const int first = start_row[e] / TILE_ROWS, n = (total[e] + TILE_ROWS - 1) / TILE_ROWS;
        for (int i = 0; i < n && first + i < max_tiles; ++i) tile_group[first + i] = e;
    }
    for (int t = used_tiles + tid; t < max_tiles; t += blockDim.x) tile_group[t] = -1;
    for (int p = p0 + lane; p < p1; p += 32) {
        const int e = ids[p];
        if (e >= 0 && e < experts && slot_of_pair[p] >= 0) slot_of_pair[p] += start_row[e] + mine[e];
    }
}

// xg[slot_of_pair[p], :] = bfloat16(weight * h[p / top, :]); a block per pair, 16 bytes per thread and turn
__global__ void __launch_bounds__(128)
moe_tile_gather_kernel(const __nv_bfloat16* __restrict__ h, const int* __restrict__ slot_of_pair, const float* __restrict__ wts,
                       int width, int top, int weight_input, __nv_bfloat16* __restrict__ xg) {
    pdl_trigger();
    pdl_wait();
    const int p = blockIdx.x;
    const int slot = slot_of_pair[p];
    if (slot < 0) return;
    const float wt = weight_input ? wts[p] : 1.0f;
    const uint4* src = reinterpret_cast<const uint4*>(h + (size_t)(p / top) * width);
    uint4* dst = reinterpret_cast<uint4*>(xg + (size_t)slot * width);
    for (int i = threadIdx.x; i < width / 8; i += blockDim.x) {
        uint4 raw = src[i];
        if (weight_input) {
            __nv_bfloat162* v = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float2 f = __bfloat1622float2(v[u]);
                v[u] = __floats2bfloat162_rn(wt * f.x, wt * f.y);
            }
        }
        dst[i] = raw;
    }
}

// out[r, :] = sum over the row's choices, in order, of out_g[slot_of_pair[r * top + k], :]  (times the weight when it
// multiplies the output), and what SumTail says; width a multiple of 4
__global__ void __launch_bounds__(256)
moe_tile_sum_kernel(const float* __restrict__ out_g, const int* __restrict__ slot_of_pair, const float* __restrict__ wts,
                    int width, int top, int weight_input, float* __restrict__ out, SumTail tail) {
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const float ew = tail.extra ? tail.extra_w[r] : 0.f;
    for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) {
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f), e = a, x = a;
        if (tail.extra) e = *reinterpret_cast<const float4*>(tail.extra + (size_t)r * width + c);
        if (tail.accumulate) x = *reinterpret_cast<const float4*>(out + (size_t)r * width + c);
        for (int k = 0; k < top; ++k) {
            const int slot = slot_of_pair[r * top + k];
            if (slot < 0) continue;
            const float wt = weight_input ? 1.0f : wts[r * top + k];
            const float4 v = *reinterpret_cast<const float4*>(out_g + (size_t)slot * width + c);
            a.x += wt * v.x; a.y += wt * v.y; a.z += wt * v.z; a.w += wt * v.w;
        }
        a.x += ew * e.x; a.y += ew * e.y; a.z += ew * e.z; a.w += ew * e.w;
        if (tail.accumulate) { a.x += x.x; a.y += x.y; a.z += x.z; a.w += x.w; }
        *reinterpret_cast<float4*>(out + (size_t)r * width + c) = a;
        if (tail.copy) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(a.x, a.y), hi = __floats2bfloat162_rn(a.z, a.w);
            *reinterpret_cast<uint2*>(tail.copy + (size_t)r * width + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo),
                                                                                      *reinterpret_cast<const uint32_t*>(&hi));
        }
    }
}

}  // namespace imparo

using namespace imparo;


// The choice's parameters (both entry points): groups, keep (experts in `groups` equal groups of neighbours, only the
// `keep` best groups' experts may be chosen; groups <= 1: all), group_pair (a group's score is the sum of its two largest
// choice scores, else its largest), correction (float32 [experts] or null: the choice goes by sigmoid(z) + correction, the
// weights by sigmoid(z); sigmoid scores only), renorm_eps (added to the chosen scores' sum before the division when renormalise
// is set), weight_scale (a factor on the weights), out_stride (ids and wts have out_stride >= top entries per row: the entries
// beyond `top` name experts every row uses with weight 1, numbered from `experts` on), extra_out (float32 [n_rows] or null:
// sigmoid of the logit column behind the experts').
static inline size_t pick_smem_bytes(int experts, int groups) {
    return (size_t)4 * (experts + (groups > 1 ? groups : 0)) * sizeof(float);
}

static inline bool pick_args_ok(int experts, int top, int groups, int keep, int out_stride, int softmax_scores, const float* correction) {
    if (pick_smem_bytes(experts, groups) > 48 * 1024) return false;
    if (top < 1 || top > experts || top > 32 || experts > 2048 || out_stride < top || out_stride > top + 32) return false;
    if (groups > 1 && (experts % groups != 0 || keep < 1 || keep > groups || keep * (experts / groups) < top)) return false;
    if (softmax_scores && correction != nullptr) return false;
    return true;
}

// logits: float32 scratch [n_rows, columns], w_r [columns, width] with columns = experts, or experts + 1 with extra_out.  Two
// launches.
extern "C" int imparo_moe_route(const void* h, int dtype, const float* w_r, int n_rows, int width, int experts, int top,
                                int softmax_scores, int renormalise, int groups, int keep, int group_pair, const float* correction,
                                float renorm_eps, float weight_scale, int out_stride, float* logits, int* ids, float* wts,
                                float* extra_out, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (!pick_args_ok(experts, top, groups, keep, out_stride, softmax_scores, correction) || logits == nullptr) return -2;
    const int columns = experts + (extra_out != nullptr ? 1 : 0);
    int per = 4;
    if ((size_t)4 * width * sizeof(float) > 48 * 1024) per = 1;
    const size_t smem = (size_t)per * width * sizeof(float);
    if (smem > 48 * 1024) return -25;
    dim3 grid((n_rows + per - 1) / per, (columns + 7) / 8);
    if (dtype == IMPARO_DT_F32)
        launch(moe_logits_kernel<float>, grid, dim3(256), smem, stream, (const float*)h, w_r, n_rows, width, columns, per, logits);
    else if (dtype == IMPARO_DT_BF16)
        launch(moe_logits_kernel<__nv_bfloat16>, grid, dim3(256), smem, stream, (const __nv_bfloat16*)h, w_r, n_rows, width, columns,
               per, logits);
    else return -1;
    IMPARO_CHECK_LAUNCH();
    launch(moe_pick_kernel, dim3((n_rows + 3) / 4), dim3(128), pick_smem_bytes(experts, groups), stream, (const float*)logits, n_rows,
           experts, columns, 1, top, softmax_scores, renormalise, groups, keep, group_pair, correction, renorm_eps, weight_scale,
           out_stride, ids, wts, extra_out);
    IMPARO_CHECK_LAUNCH();
    return 0;
}

// The choice alone, from logits that a product has made: [n_rows, parts * columns] float32 (columns >= experts, or >= experts + 1
// with extra_out; more pad the product's width).  With bfloat16 rows h (exact in 32-bit) and the 32-bit router matrix cut into three bfloat16 pieces (w1 = W
// rounded, w2 = W - w1 rounded, w3 the rest rounded: 8 + 8 + 8 bits of mantissa, their sum is W to its last bit), the
// tensor-core product h [w1; w2; w3]^T has exact products and 32-bit sums: the router's logits in 32-bit, at the product's speed.
extern "C" int imparo_moe_pick(const float* logits, int n_rows, int experts, int columns, int parts, int top, int softmax_scores, int renormalise,
                               int groups, int keep, int group_pair, const float* correction, float renorm_eps, float weight_scale,
                               int out_stride, int* ids, float* wts, float* extra_out, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (!pick_args_ok(experts, top, groups, keep, out_stride, softmax_scores, correction) || parts < 1 || parts > 4
        || columns < experts + (extra_out != nullptr ? 1 : 0)) return -2;
    launch(moe_pick_kernel, dim3((n_rows + 3) / 4), dim3(128), pick_smem_bytes(experts, groups), stream, logits, n_rows, experts,
           columns, parts, top, softmax_scores, renormalise, groups, keep, group_pair, correction,
           renorm_eps, weight_scale, out_stride, ids, wts, extra_out);
    IMPARO_CHECK_LAUNCH();
    return 0;
}

constexpr size_t FEW_SMEM_MOST = 200 * 1024;

template <typename T, bool UP>
static int few_launch(const void* in, const void* w, const int* ids, const float* wts, int n_rows, int n, int n_feat, int top, int experts,
                      int weight_input, int gated, int act, float limit, void* out, const SharedRows& sh, cudaStream_t stream) {
    const int rows = FEW_ROWS, pairs = n_rows * top;
    if constexpr (sizeof(T) == 2) {
        uintptr_t all = (uintptr_t)in | (uintptr_t)w | (uintptr_t)sh.w | (uintptr_t)sh.in;
        if (n % 8 == 0 && (sh.w == nullptr || sh.n % 8 == 0) && (all & 15) == 0) {
            const int nb = n_rows > 8 ? 2 : 1, per = gated ? 8 : 16;
            int st = (n_feat + per - 1) / per, tl = 0;
            if (sh.w) {
                st = st > (sh.n_feat + 15) / 16 ? st : (sh.n_feat + 15) / 16;
                tl = (n_rows + 8 * nb - 1) / (8 * nb);
            }
            const dim3 grid(tl + (pairs < experts ? pairs : experts), st), block(MM_WARPS * 32);
            if (st > 65535) return -2;
            if (nb == 1) launch(moe_few_mma_kernel<UP, 1>, grid, block, 0, stream, (const T*)in, (const T*)w, ids, wts, n_rows, n, n_feat, top,
                                experts, weight_input, gated, act, limit, out, sh);
            else launch(moe_few_mma_kernel<UP, 2>, grid, block, 0, stream, (const T*)in, (const T*)w, ids, wts, n_rows, n, n_feat, top, experts,
                        weight_input, gated, act, limit, out, sh);
            IMPARO_CHECK_LAUNCH();
            return 0;
        }
    }
    size_t smem = (size_t)(pairs < rows ? pairs : rows) * n * sizeof(T);
    int stretches = (n_feat + (gated ? 15 : 31)) / (gated ? 16 : 32), tiles = 0;
    if (sh.w) {
        const size_t b = (size_t)(n_rows < rows ? n_rows : rows) * sh.n * sizeof(T);
        smem = smem > b ? smem : b;
        stretches = stretches > (sh.n_feat + 31) / 32 ? stretches : (sh.n_feat + 31) / 32;
        tiles = (n_rows + FEW_ROWS - 1) / FEW_ROWS;
    }
    if (smem > FEW_SMEM_MOST) return -25;
    static size_t allowed = 44 * 1024;                     // (a few KB beside it are the kernel's own)
    if (smem > allowed) {
        const cudaError_t e = cudaFuncSetAttribute(moe_few_kernel<T, UP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)FEW_SMEM_MOST);
        if (e != cudaSuccess) return (int)e;
        allowed = FEW_SMEM_MOST;
    }
    launch(moe_few_kernel<T, UP>, dim3(tiles + (pairs < experts ? pairs : experts), stretches), dim3(256), smem, stream, (const T*)in, (const T*)w,
           ids, wts, n_rows, n, n_feat, top, experts, weight_input, gated, act, limit, out, sh);
    IMPARO_CHECK_LAUNCH();
    return 0;
}

extern "C" int imparo_moe_sum(const float* pair_out, int n_rows, int width, int top, const float* extra, const float* extra_w,
                              int accumulate, float* out, void* copy, cudaStream_t stream);

// gated = 1: w_gu [experts, 2 ff, width], act one of gated_act's kinds (with limit); gated = 0: w_gu [experts, ff, width], act one
// of plain_act's.  mid: [n_rows * top, ff] in dtype; pair_out float32 [n_rows * top, width]; out float32 [n_rows, width].  With s_up
// (needs gated = 0): an expert that every row uses, s_up [s_ff, width] and s_down [width, s_ff], runs in the same launches: s_mid
// [n_rows, s_ff] in dtype, s_out float32 [n_rows, width] receives its output, unweighted.  extra, extra_w, accumulate, copy as for
// imparo_moe_sum (extra may be s_out).  Three launches per 256 pairs.  -25: rows too wide for eight of them in shared memory.
extern "C" int imparo_moe_rows(const void* h, const void* w_gu, const void* w_down, int dtype, const int* ids, const float* wts,
                               int n_rows, int width, int ff, int top, int experts, int weight_input, int gated, int act, float limit,
                               void* mid, float* pair_out, const void* s_up, const void* s_down, int s_ff, void* s_mid, float* s_out,
                               const float* extra, const float* extra_w, int accumulate, float* out, void* copy, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (top < 1 || top > FEW_PAIRS || width < 1 || ff < 1) return -2;
    if (s_up != nullptr && (gated || s_down == nullptr || s_ff < 1 || s_mid == nullptr || s_out == nullptr)) return -2;
    if (dtype != IMPARO_DT_F32 && dtype != IMPARO_DT_BF16) return -1;
    const size_t elt = dtype == IMPARO_DT_F32 ? 4 : 2;
    const int step = FEW_PAIRS / top;
    for (int r0 = 0; r0 < n_rows; r0 += step) {
        const int rows = n_rows - r0 < step ? n_rows - r0 : step;
        const size_t p0 = (size_t)r0 * top;
        const char* hr = (const char*)h + (size_t)r0 * width * elt;
        char* mr = (char*)mid + p0 * ff * elt;
        SharedRows up = {}, down = {};
        if (s_up != nullptr) {
            char* sm = (char*)s_mid + (size_t)r0 * s_ff * elt;
            up = {s_up, hr, sm, s_ff, width};
            down = {s_down, sm, s_out + (size_t)r0 * width, width, s_ff};
        }
        int rc;
        if (dtype == IMPARO_DT_F32) {
            rc = few_launch<float, true>(hr, w_gu, ids + p0, wts + p0, rows, width, ff, top, experts, weight_input, gated, act, limit, mr, up, stream);
            if (rc == 0) rc = few_launch<float, false>(mr, w_down, ids + p0, wts + p0, rows, ff, width, top, experts, weight_input, 0, 0, 0.f,
                                                       pair_out + p0 * width, down, stream);
        } else {
            rc = few_launch<__nv_bfloat16, true>(hr, w_gu, ids + p0, wts + p0, rows, width, ff, top, experts, weight_input, gated, act, limit, mr, up,
                                                 stream);
            if (rc == 0) rc = few_launch<__nv_bfloat16, false>(mr, w_down, ids + p0, wts + p0, rows, ff, width, top, experts, weight_input, 0, 0, 0.f,
                                                               pair_out + p0 * width, down, stream);
        }
        if (rc) return rc;
    }
    return imparo_moe_sum(pair_out, n_rows, width, top, extra, extra_w, accumulate, out, copy, stream);
}

// out[r, :] = (accumulate: its old value +) sum_k pair_out[r * top + k, :] (+ extra_w[r] * extra[r, :]); copy: the result rounded
// to bfloat16, or null.
extern "C" int imparo_moe_sum(const float* pair_out, int n_rows, int width, int top, const float* extra, const float* extra_w,
                              int accumulate, float* out, void* copy, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (top < 0 || (extra != nullptr && extra_w == nullptr)) return -2;
    const SumTail tail = {extra, extra_w, accumulate, (__nv_bfloat16*)copy};
    const bool vec = width % 4 == 0 && (((uintptr_t)pair_out | (uintptr_t)extra | (uintptr_t)out | (uintptr_t)copy) & 15) == 0;
    const size_t total = (size_t)n_rows * width / (vec ? 4 : 1);
    const dim3 grid((unsigned)((total + 255) / 256 > 4096 ? 4096 : (total + 255) / 256));
    if (vec) launch(moe_sum_pairs_kernel<true>, grid, dim3(256), 0, stream, pair_out, n_rows, width, top, out, tail);
    else launch(moe_sum_pairs_kernel<false>, grid, dim3(256), 0, stream, pair_out, n_rows, width, top, out, tail);
    IMPARO_CHECK_LAUNCH();
    return 0;
}

// scratch_i: int32 [n_pairs + experts + 1 + 1 + 3 * max_tiles], max_tiles = n_pairs / 32 + experts; pair_out float32
// [n_pairs, width]; mid [n_pairs, ff] in dtype; out float32 [n_rows, width]; gated, act, limit as above; extra, extra_w,
// accumulate, copy as for imparo_moe_sum.  Four launches.
extern "C" int imparo_moe_grouped(const void* h, const void* w_gu, const void* w_down, int dtype, const int* ids, const float* wts,
                                  int n_rows, int width, int ff, int top, int experts, int weight_input, int gated, int act,
                                  float limit, void* mid, float* pair_out, int* scratch_i, const float* extra, const float* extra_w,
                                  int accumulate, float* out, void* copy, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    const int n_pairs = n_rows * top;
    const int max_tiles = n_pairs / GM + experts;
    if (experts > 4096) return -25;
    int* sorted = scratch_i;
    int* expert_start = scratch_i + n_pairs;
    int* plan = expert_start + experts + 1;
    launch(moe_group_plan_kernel, dim3(1), dim3(1024), (size_t)(experts + 1) * sizeof(int), stream, ids, n_pairs, experts, sorted,
           expert_start, plan, max_tiles);
    IMPARO_CHECK_LAUNCH();
    dim3 g1(max_tiles, (ff + GN - 1) / GN), g2(max_tiles, (width + GN - 1) / GN);
    if (dtype == IMPARO_DT_F32) {
        launch(moe_group_up_kernel<float>, g1, dim3(256), 0, stream, (const float*)h, (const float*)w_gu, (const int*)sorted,
               (const int*)plan, wts, width, ff, top, weight_input, gated, act, limit, (float*)mid);
        IMPARO_CHECK_LAUNCH();
        launch(moe_group_down_kernel<float>, g2, dim3(256), 0, stream, (const float*)mid, (const float*)w_down, (const int*)sorted,
               (const int*)plan, wts, width, ff, weight_input, pair_out);
    } else if (dtype == IMPARO_DT_BF16) {
        launch(moe_group_up_kernel<__nv_bfloat16>, g1, dim3(256), 0, stream, (const __nv_bfloat16*)h, (const __nv_bfloat16*)w_gu,
               (const int*)sorted, (const int*)plan, wts, width, ff, top, weight_input, gated, act, limit, (__nv_bfloat16*)mid);
        IMPARO_CHECK_LAUNCH();
        launch(moe_group_down_kernel<__nv_bfloat16>, g2, dim3(256), 0, stream, (const __nv_bfloat16*)mid, (const __nv_bfloat16*)w_down,
               (const int*)sorted, (const int*)plan, wts, width, ff, weight_input, pair_out);
    } else return -1;
    IMPARO_CHECK_LAUNCH();
    return imparo_moe_sum(pair_out, n_rows, width, top, extra, extra_w, accumulate, out, copy, stream);
}

extern "C" int imparo_gemm_prefill_grouped(const void* x, int ldx, const void* w, int n_groups, void* out, int ldo, int m_tiles,
                                           int N, int K, int epilogue, int act, float limit, const int* tile_group, int* status,
                                           cudaStream_t stream);

// bfloat16, width and ff multiples of 8, at most 256 experts: rows sorted into tiles of 128 per expert and both products on
// the tensor-memory kernel (the activation in the first one's epilogue).  m_tiles = n_pairs / 128 + experts; xg bfloat16
// [m_tiles * 128, width]; mid_g bfloat16 [m_tiles * 128, ff]; out_g float32 [m_tiles * 128, width]; scratch_i int32
// [n_pairs + m_tiles]; out float32 [n_rows, width]; gated, act, limit, extra, extra_w, accumulate, copy as above.  Five launches.
// -25: not a case for this path.
extern "C" int imparo_moe_tiles(const void* h, const void* w_gu, const void* w_down, const int* ids, const float* wts, int n_rows,
                                int width, int ff, int top, int experts, int weight_input, int gated, int act, float limit, void* xg,
                                void* mid_g, float* out_g, int* scratch_i, const float* extra, const float* extra_w, int accumulate,
                                float* out, void* copy, int* status, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width % 8 != 0 || ff % 8 != 0 || experts > 256) return -25;
    if (extra != nullptr && extra_w == nullptr) return -2;
    const int n_pairs = n_rows * top;
    const int m_tiles = n_pairs / TILE_ROWS + experts;
    int* slot_of_pair = scratch_i;
    int* tile_group = scratch_i + n_pairs;
    launch(moe_tile_plan_kernel, dim3(1), dim3(1024), (size_t)34 * experts * sizeof(int), stream, ids, n_pairs, experts, slot_of_pair,
           tile_group, m_tiles);
    IMPARO_CHECK_LAUNCH();
    launch(moe_tile_gather_kernel, dim3(n_pairs), dim3(128), 0, stream, (const __nv_bfloat16*)h, (const int*)slot_of_pair, wts, width,
           top, weight_input, (__nv_bfloat16*)xg);
    IMPARO_CHECK_LAUNCH();
    int rc = imparo_gemm_prefill_grouped(xg, width, w_gu, experts, mid_g, ff, m_tiles, ff, width, gated ? 3 : 4, act, limit, tile_group,
                                         status, stream);
    if (rc) return rc;
    rc = imparo_gemm_prefill_grouped(mid_g, ff, w_down, experts, out_g, width, m_tiles, width, ff, 1, 0, 0.f, tile_group, status, stream);
    if (rc) return rc;
    const SumTail tail = {extra, extra_w, accumulate, (__nv_bfloat16*)copy};
    launch(moe_tile_sum_kernel, dim3(n_rows), dim3(256), 0, stream, (const float*)out_g, (const int*)slot_of_pair, wts, width, top,
           weight_input, out, tail);
    IMPARO_CHECK_LAUNCH();
    return 0;
}
