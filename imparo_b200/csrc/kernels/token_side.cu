// A layer's own token input: from the stream x (32-bit) and the token's stretch e of a side table,
//   g = gelu(G x) * e,  gelu(z) = 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))),
// which a product P g and a normed add (group_norm.cu) bring back into the stream.
//
//  (1) token_side_gate: few rows.  A warp per entry of g and up to eight rows: the row of G is read once for them, x as it
//      stands in 32-bit, the sums are 32-bit; activation and side entry in the same launch.
//  (2) token_side_act: many rows, from a product's 32-bit rows G x.
#include "common.cuh"

namespace imparo {
namespace ts {

constexpr int ROWS = 8, WARPS = 4;

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
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, j = blockIdx.x * WARPS + (threadIdx.x >> 5);
    const int r0 = blockIdx.y * ROWS, R = min(ROWS, n_rows - r0);
    if (j >= dim) return;
    const T* wr = w + (size_t)j * width;
    const float* xr = x + (size_t)r0 * width;
    float acc[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) acc[r] = 0.f;
    const bool vec = width % 8 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0;
    if (vec) {
        for (int i = lane * 8; i < width; i += 256) {
            float wv[8];
            if constexpr (sizeof(T) == 2) {
                const uint4 raw = *reinterpret_cast<const uint4*>(wr + i);
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const float2 f = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&raw)[u]);
                    wv[2 * u] = f.x;
                    wv[2 * u + 1] = f.y;
                }
            } else {
#pragma unroll
                for (int u = 0; u < 8; ++u) wv[u] = to_f32(wr[i + u]);
            }
            float4 a[ROWS], b[ROWS];                       // every row's entries in flight at once
#pragma unroll
            for (int r = 0; r < ROWS; ++r)
                if (r < R) {
                    a[r] = *reinterpret_cast<const float4*>(xr + (size_t)r * width + i);
                    b[r] = *reinterpret_cast<const float4*>(xr + (size_t)r * width + i + 4);
                }
#pragma unroll
            for (int r = 0; r < ROWS; ++r)
                if (r < R)
                    acc[r] += (wv[0] * a[r].x + wv[1] * a[r].y) + (wv[2] * a[r].z + wv[3] * a[r].w)
                              + ((wv[4] * b[r].x + wv[5] * b[r].y) + (wv[6] * b[r].z + wv[7] * b[r].w));
        }
    } else {
        for (int i = lane; i < width; i += 32) {
            const float wv = to_f32(wr[i]);
#pragma unroll
            for (int r = 0; r < ROWS; ++r) if (r < R) acc[r] += wv * xr[(size_t)r * width + i];
        }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) acc[r] = warp_sum(acc[r]);
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        if (lane == r && r < R) {
            const int id = side_token(ids, rows, r0 + r, vocab, status);
            const float e = id < 0 ? 0.f : to_f32(table[(size_t)id * table_stride + col0 + j]);
            out[(size_t)(r0 + r) * dim + j] = from_f32<T>(gelu_times<T>(acc[r], e));
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256)
side_act_kernel(const float* __restrict__ z, const T* __restrict__ table, size_t table_stride, int col0, const int* __restrict__ ids,
                const int* __restrict__ rows, int n_rows, int dim, int vocab, T* __restrict__ out, int* status) {
    pdl_trigger();
    pdl_wait();
    const size_t total = (size_t)n_rows * dim;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const int r = (int)(i / dim), j = (int)(i - (size_t)r * dim);
        const int id = side_token(ids, rows, r, vocab, status);
        const float e = id < 0 ? 0.f : to_f32(table[(size_t)id * table_stride + col0 + j]);
        out[i] = from_f32<T>(gelu_times<T>(z[i], e));
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
    const dim3 grid((dim + ts::WARPS - 1) / ts::WARPS, tiles), block(ts::WARPS * 32);
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
    const size_t total = (size_t)n_rows * dim;
    const dim3 grid((unsigned)((total + 255) / 256 > 8192 ? 8192 : (total + 255) / 256));
    if (dtype == IMPARO_DT_F32)
        launch(ts::side_act_kernel<float>, grid, dim3(256), 0, stream, z, (const float*)table, (size_t)table_stride, col0, ids, rows,
               n_rows, dim, vocab, (float*)out, status);
    else if (dtype == IMPARO_DT_BF16)
        launch(ts::side_act_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, z, (const __nv_bfloat16*)table, (size_t)table_stride, col0,
               ids, rows, n_rows, dim, vocab, (__nv_bfloat16*)out, status);
    else return -1;
    IMPARO_CHECK_LAUNCH();
    return 0;
}
