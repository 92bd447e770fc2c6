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
#include "common.cuh"

namespace imparo {
namespace gla {

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

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
