// A layer's own token input: from the stream x (32-bit) and the token's stretch e of a side table,
//   g = gelu(G x) * e,  gelu(z) = 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))),
// which a product P g and a normed add (group_norm.cu) bring back into the stream.
//
//  (1) token_side_gate: few rows.  A block per two entries of g and up to eight rows, its warps splitting the width: the rows of G
//      are read once for them, x as it stands in 32-bit, the sums are 32-bit in a fixed order; activation and side entry in the same
//      launch.
//  (2) token_side_act: many rows, from a product's 32-bit rows G x.
#include "common.cuh"

namespace imparo {
namespace ts {

constexpr int ROWS = 8, WARPS = 8, FEATS = 2;

// the side table's row of a step's row: rows (int32, or null) names which of the step's tokens row r of x is
__device__ __forceinline__ int side_token(const int* __restrict__ ids, const int* __restrict__ rows, int r, int vocab, int* status) {
    const int t = rows ? rows[r] : r;
    const int id = ids[t];
    if (id < 0 || id >= vocab) {
        report(status, IMPARO_ST_TOKEN_RANGE, 90, t, id);
        return -1;
    }
    return id;
}

template <typename T>
__device__ __forceinline__ float gelu_times(float z, float e) {
    return (sizeof(T) == 2 ? plain_act_bf16(1, z) : plain_act(1, z)) * e;
}

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
side_gate_kernel(const float* __restrict__ x, const T* __restrict__ w, const T* __restrict__ table, size_t table_stride, int col0,
                 const int* __restrict__ ids, const int* __restrict__ rows, int n_rows, int width, int dim, int vocab,
                 T* __restrict__ out, int* status) {
    __shared__ float part[WARPS][FEATS * ROWS];
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, j0 = blockIdx.x * FEATS;
    const int r0 = blockIdx.y * ROWS, R = min(ROWS, n_rows - r0);
    const float* xr = x + (size_t)r0 * width;
    float acc[FEATS][ROWS];
#pragma unroll
    for (int f = 0; f < FEATS; ++f)
#pragma unroll
        for (int r = 0; r < ROWS; ++r) acc[f][r] = 0.f;
    pdl_wait();
    const bool vec = width % 4 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0;
    if (vec) {
        for (int i = (warp * 32 + lane) * 4; i < width; i += WARPS * 128) {
            float wv[FEATS][4];
#pragma unroll
            for (int f = 0; f < FEATS; ++f) {
                if (j0 + f >= dim) { wv[f][0] = wv[f][1] = wv[f][2] = wv[f][3] = 0.f; continue; }
                const T* wr = w + (size_t)(j0 + f) * width + i;
                if constexpr (sizeof(T) == 2) {
                    const uint2 raw = *reinterpret_cast<const uint2*>(wr);
                    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
                    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
                    wv[f][0] = lo.x; wv[f][1] = lo.y; wv[f][2] = hi.x; wv[f][3] = hi.y;
                } else {
                    const float4 v = *reinterpret_cast<const float4*>(wr);
                    wv[f][0] = v.x; wv[f][1] = v.y; wv[f][2] = v.z; wv[f][3] = v.w;
                }
            }
            float4 a[ROWS];                               // every row's entries in flight at once
#pragma unroll
            for (int r = 0; r < ROWS; ++r) if (r < R) a[r] = *reinterpret_cast<const float4*>(xr + (size_t)r * width + i);
#pragma unroll
            for (int r = 0; r < ROWS; ++r)
                if (r < R) {
#pragma unroll
                    for (int f = 0; f < FEATS; ++f) acc[f][r] += (wv[f][0] * a[r].x + wv[f][1] * a[r].y) + (wv[f][2] * a[r].z + wv[f][3] * a[r].w);
                }
        }
    } else {
        for (int i = threadIdx.x; i < width; i += WARPS * 32) {
#pragma unroll
            for (int f = 0; f < FEATS; ++f) {
                if (j0 + f >= dim) continue;
                const float wv = to_f32(w[(size_t)(j0 + f) * width + i]);
#pragma unroll
                for (int r = 0; r < ROWS; ++r) if (r < R) acc[f][r] += wv * xr[(size_t)r * width + i];
            }
        }
    }
#pragma unroll
    for (int f = 0; f < FEATS; ++f)
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const float v = warp_sum(acc[f][r]);
            if (lane == 0) part[warp][f * ROWS + r] = v;
        }
    __syncthreads();
    if (threadIdx.x < FEATS * ROWS) {
        const int f = threadIdx.x / ROWS, r = threadIdx.x % ROWS, j = j0 + f;
        if (r < R && j < dim) {
            float z = 0.f;
#pragma unroll
            for (int k = 0; k < WARPS; ++k) z += part[k][threadIdx.x];
            const int id = side_token(ids, rows, r0 + r, vocab, status);
            const float e = id < 0 ? 0.f : to_f32(table[(size_t)id * table_stride + col0 + j]);
            out[(size_t)(r0 + r) * dim + j] = from_f32<T>(gelu_times<T>(z, e));
        }
    }
}

// VEC: four entries at a time (dim, col0 and the table's rows in multiples of 4, aligned pointers)
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
side_act_kernel(const float* __restrict__ z, const T* __restrict__ table, size_t table_stride, int col0, const int* __restrict__ ids,
                const int* __restrict__ rows, int n_rows, int dim, int vocab, T* __restrict__ out, int* status) {
    constexpr int N = VEC ? 4 : 1;
    pdl_trigger();
    pdl_wait();
    const int per = dim / N;
    const size_t total = (size_t)n_rows * per;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const int r = (int)(i / per), j = (int)(i - (size_t)r * per) * N;
        const int id = side_token(ids, rows, r, vocab, status);
        struct alignas(sizeof(T) * N) Some { T v[N]; } e, o;
        if (id >= 0) {
            e = *reinterpret_cast<const Some*>(table + (size_t)id * table_stride + col0 + j);
        } else {
#pragma unroll
            for (int u = 0; u < N; ++u) e.v[u] = from_f32<T>(0.f);
        }
        struct alignas(4 * N) Row { float v[N]; };
        const Row zv = *reinterpret_cast<const Row*>(z + (size_t)r * dim + j);
#pragma unroll
        for (int u = 0; u < N; ++u) o.v[u] = from_f32<T>(gelu_times<T>(zv.v[u], to_f32(e.v[u])));
        *reinterpret_cast<Some*>(out + (size_t)r * dim + j) = o;
    }
}

}  // namespace ts
}  // namespace imparo

using namespace imparo;

// out [n_rows, dim] = gelu(x w^T) * table[ids[rows[r]], col0 : col0 + dim] (rows null: row r is token r); x float32
// [n_rows, width], w [dim, width], table [vocab, table_stride] and out in dtype.
extern "C" int imparo_token_side_gate(const float* x, const void* w, const void* table, long long table_stride, int col0, int dtype,
                                      const int* ids, const int* rows, int n_rows, int width, int dim, int vocab, void* out,
                                      int* status, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width < 1 || dim < 1 || col0 < 0 || col0 + dim > table_stride) return -2;
    const int tiles = (n_rows + ts::ROWS - 1) / ts::ROWS;
    if (tiles > 65535) return -2;
    const dim3 grid((dim + ts::FEATS - 1) / ts::FEATS, tiles), block(ts::WARPS * 32);
    if (dtype == IMPARO_DT_F32)
        launch(ts::side_gate_kernel<float>, grid, block, 0, stream, x, (const float*)w, (const float*)table, (size_t)table_stride, col0,
               ids, rows, n_rows, width, dim, vocab, (float*)out, status);
    else if (dtype == IMPARO_DT_BF16)
        launch(ts::side_gate_kernel<__nv_bfloat16>, grid, block, 0, stream, x, (const __nv_bfloat16*)w, (const __nv_bfloat16*)table,
               (size_t)table_stride, col0, ids, rows, n_rows, width, dim, vocab, (__nv_bfloat16*)out, status);
    else return -1;
    IMPARO_CHECK_LAUNCH();
    return 0;
}

// The same from the product's rows z = x w^T, float32 [n_rows, dim].
extern "C" int imparo_token_side_act(const float* z, const void* table, long long table_stride, int col0, int dtype, const int* ids,
                                     const int* rows, int n_rows, int dim, int vocab, void* out, int* status, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (dim < 1 || col0 < 0 || col0 + dim > table_stride) return -2;
    const bool vec = dim % 4 == 0 && col0 % 4 == 0 && table_stride % 4 == 0 && (((uintptr_t)z | (uintptr_t)table | (uintptr_t)out) & 15) == 0;
    const size_t total = (size_t)n_rows * dim / (vec ? 4 : 1);
    const dim3 grid((unsigned)((total + 255) / 256 > 8192 ? 8192 : (total + 255) / 256));
#define IMPARO_TSA(T_, V_) launch(ts::side_act_kernel<T_, V_>, grid, dim3(256), 0, stream, z, (const T_*)table, (size_t)table_stride, col0, \
        ids, rows, n_rows, dim, vocab, (T_*)out, status)
    if (dtype == IMPARO_DT_F32) { if (vec) IMPARO_TSA(float, true); else IMPARO_TSA(float, false); }
    else if (dtype == IMPARO_DT_BF16) { if (vec) IMPARO_TSA(__nv_bfloat16, true); else IMPARO_TSA(__nv_bfloat16, false); }
    else return -1;
#undef IMPARO_TSA
    IMPARO_CHECK_LAUNCH();
    return 0;
}
