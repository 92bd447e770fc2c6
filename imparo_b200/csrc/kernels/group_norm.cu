// RMS norm in groups, and the residual add of a normed sublayer output.
//
// The row is cut into `groups` equal consecutive stretches, each divided by its own root mean square (sqrt(mean of the
// stretch's squares + eps), eps inside the root); the whole row is then multiplied by a weight.  groups = 1 is the plain
// RMS norm.
//
//  (1) group_rmsnorm:  out[r] = gnorm(x[rows[r]]) * w
//  (2) group_norm_add: x[r] += gnorm(y[r]) * wb, and in the same pass, when out is given, out[r] = gnorm(x[r]) * wn of the
//      updated row: the norm after one sublayer, its add into the 32-bit stream and the norm before the next sublayer.
//      y may still be the split partials of the product that makes it (summed in split order) and may lack its bias.
//
// Few rows: a block per row.  A group belongs to a team of `wpg` warps (one warp per group when there are at least as many groups as
// warps); the sum over a group is a fixed tree over the team's lanes, so a row's result depends on the row alone.
// Many rows (a prompt portion) with groups of up to 4,096 elements: one, two or four warps per (row, group) that keep the group in
// registers; every load of the group is in flight at once.  All arithmetic is 32-bit.
#include "common.cuh"

namespace imparo {
namespace gn {

constexpr int MAX_WARPS = 16;
constexpr int REGS = 4;             // vectors of a group that a thread keeps in registers; longer groups are read again

template <typename TOut, int V> struct Vec;
template <typename TOut> struct Vec<TOut, 1> {
    float v[1];
    __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
    __device__ __forceinline__ void load_cg(const float* p) { v[0] = __ldcg(p); }
    __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
    static __device__ __forceinline__ void put(TOut* p, const float (&o)[1]) { *p = from_f32<TOut>(o[0]); }
};
template <typename TOut> struct Vec<TOut, 4> {
    float v[4];
    __device__ __forceinline__ void load(const float* p) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    }
    __device__ __forceinline__ void load_cg(const float* p) {
        const float4 q = __ldcg(reinterpret_cast<const float4*>(p));
        v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    }
    __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    static __device__ __forceinline__ void put(TOut* p, const float (&o)[4]) {
        if (sizeof(TOut) == 4) {
            *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]);
        } else {
            const __nv_bfloat162 a = __floats2bfloat162_rn(o[0], o[1]), b = __floats2bfloat162_rn(o[2], o[3]);
            *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
        }
    }
};

// sum over the team's warps; every thread of the block calls it (the barriers are the block's)
__device__ __forceinline__ float team_sum(float v, float* scratch, int wpg) {
    v = warp_sum(v);
    if (wpg == 1) return v;
    const int warp = threadIdx.x >> 5;
    __syncthreads();
    if ((threadIdx.x & 31) == 0) scratch[warp] = v;
    __syncthreads();
    float s = 0.f;
    const int first = warp / wpg * wpg;
    for (int i = 0; i < wpg; ++i) s += first + i < MAX_WARPS ? scratch[first + i] : 0.f;
    return s;
}

template <typename TOut, int V>
__global__ void group_rmsnorm_kernel(const float* __restrict__ x, const int* __restrict__ rows, const float* __restrict__ w,
                                     float eps, TOut* __restrict__ out, int width, int groups, int wpg) {
    using W = Vec<TOut, V>;
    __shared__ float scratch[MAX_WARPS];
    if (threadIdx.x < MAX_WARPS) scratch[threadIdx.x] = 0.f;
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float* xr = x + (size_t)(rows ? rows[r] : r) * width;
    const int gw = width / groups, teams = (int)(blockDim.x >> 5) / wpg, team = warp / wpg;
    const int at = ((warp % wpg) * 32 + lane) * V, step = wpg * 32 * V;
    for (int g0 = 0; g0 < groups; g0 += teams) {
        const int g = g0 + team;
        const bool mine = team < teams && g < groups;
        const float* xg = xr + (size_t)g * gw;
        W v[REGS];
        float ss = 0.f;
        if (mine) {
#pragma unroll
            for (int k = 0; k < REGS; ++k) {
                if (at + k * step < gw) {
                    v[k].load(xg + at + k * step);
#pragma unroll
                    for (int e = 0; e < V; ++e) ss += v[k].v[e] * v[k].v[e];
                }
            }
            for (int i = at + REGS * step; i < gw; i += step) {
                W t;
                t.load(xg + i);
#pragma unroll
                for (int e = 0; e < V; ++e) ss += t.v[e] * t.v[e];
            }
        }
        ss = team_sum(ss, scratch, wpg);
        if (!mine) continue;
        const float scale = 1.0f / sqrtf(ss / (float)gw + eps);
        auto write = [&](int i, const W& t) {
            W wv;
            wv.load(w + (size_t)g * gw + i);
            float o[V];
#pragma unroll
            for (int e = 0; e < V; ++e) o[e] = t.v[e] * scale * wv.v[e];
            W::put(out + (size_t)r * width + (size_t)g * gw + i, o);
        };
#pragma unroll
        for (int k = 0; k < REGS; ++k)
            if (at + k * step < gw) write(at + k * step, v[k]);
        for (int i = at + REGS * step; i < gw; i += step) {
            W t;
            t.load(xg + i);
            write(i, t);
        }
    }
}

template <typename TOut, int V>
__global__ void group_norm_add_kernel(float* __restrict__ x, const float* __restrict__ y, int parts, size_t part_stride,
                                      const float* __restrict__ ybias, const float* __restrict__ wb, float eps_b,
                                      const float* __restrict__ wn, float eps_n, TOut* __restrict__ out, int width, int groups,
                                      int wpg) {
    using W = Vec<TOut, V>;
    __shared__ float scratch[MAX_WARPS];
    if (threadIdx.x < MAX_WARPS) scratch[threadIdx.x] = 0.f;
    pdl_trigger();
    const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int gw = width / groups, teams = (int)(blockDim.x >> 5) / wpg, team = warp / wpg;
    const int at = ((warp % wpg) * 32 + lane) * V, step = wpg * 32 * V;
    pdl_wait();
    for (int g0 = 0; g0 < groups; g0 += teams) {
        const int g = g0 + team;
        const bool mine = team < teams && g < groups;
        const size_t row = (size_t)r * width + (size_t)g * gw, col = (size_t)g * gw;
        auto sub = [&](int i) {                              // the sublayer's output: bias, then the partials in split order
            W t;
            if (ybias) {
                t.load(ybias + col + i);
            } else {
#pragma unroll
                for (int e = 0; e < V; ++e) t.v[e] = 0.f;
            }
            for (int s0 = 0; s0 < parts; s0 += 8) {            // eight partials' loads in flight, added in order
                W p[8];
#pragma unroll
                for (int u = 0; u < 8; ++u) if (s0 + u < parts) p[u].load_cg(y + (size_t)(s0 + u) * part_stride + row + i);
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    if (s0 + u < parts) {
#pragma unroll
                        for (int e = 0; e < V; ++e) t.v[e] += p[u].v[e];
                    }
                }
            }
            return t;
        };
        W v[REGS], xv[REGS];
        float ss = 0.f;
        if (mine) {
#pragma unroll
            for (int k = 0; k < REGS; ++k) {
                if (at + k * step < gw) {
                    xv[k].load(x + row + at + k * step);
                    v[k] = sub(at + k * step);
#pragma unroll
                    for (int e = 0; e < V; ++e) ss += v[k].v[e] * v[k].v[e];
                }
            }
            for (int i = at + REGS * step; i < gw; i += step) {
                const W t = sub(i);
#pragma unroll
                for (int e = 0; e < V; ++e) ss += t.v[e] * t.v[e];
            }
        }
        ss = team_sum(ss, scratch, wpg);
        const float scale = 1.0f / sqrtf(ss / (float)gw + eps_b);
        float ss2 = 0.f;
        if (mine) {
            auto update = [&](int i, const W& t, W& xx) {
                W wv;
                wv.load(wb + col + i);
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    xx.v[e] += t.v[e] * scale * wv.v[e];
                    ss2 += xx.v[e] * xx.v[e];
                }
                xx.store(x + row + i);
            };
#pragma unroll
            for (int k = 0; k < REGS; ++k)
                if (at + k * step < gw) update(at + k * step, v[k], xv[k]);
            for (int i = at + REGS * step; i < gw; i += step) {
                W xx;
                xx.load(x + row + i);
                update(i, sub(i), xx);
            }
        }
        if (out == nullptr) continue;
        ss2 = team_sum(ss2, scratch, wpg);
        if (!mine) continue;
        const float nscale = 1.0f / sqrtf(ss2 / (float)gw + eps_n);
        auto write = [&](int i, const W& t) {
            W wv;
            wv.load(wn + col + i);
            float o[V];
#pragma unroll
            for (int e = 0; e < V; ++e) o[e] = t.v[e] * nscale * wv.v[e];
            W::put(out + row + i, o);
        };
#pragma unroll
        for (int k = 0; k < REGS; ++k)
            if (at + k * step < gw) write(at + k * step, xv[k]);
        for (int i = at + REGS * step; i < gw; i += step) {      // (this thread's own writes)
            W t;
            t.load(x + row + i);
            write(i, t);
        }
    }
}

// ---- many rows: WPG warps per (row, group), NV float4 per lane (groups of up to 128 * NV * WPG elements, multiples of 4) -------
constexpr int ROW_WARPS = 4, MANY_ROWS = 256;

// sum over a team of WPG warps (every thread of the block calls it; scratch: a float per warp, one array per sum of the kernel)
template <int WPG>
__device__ __forceinline__ float rows_team_sum(float v, float* scratch) {
    v = warp_sum(v);
    if (WPG == 1) return v;
    const int warp = threadIdx.x >> 5;
    if ((threadIdx.x & 31) == 0) scratch[warp] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < WPG; ++i) s += scratch[warp / WPG * WPG + i];
    return s;
}

template <typename TOut, int NV, int WPG>
__global__ void __launch_bounds__(ROW_WARPS * 32)
group_rmsnorm_rows_kernel(const float* __restrict__ x, const int* __restrict__ rows, const float* __restrict__ w, float eps,
                          TOut* __restrict__ out, int n_rows, int width, int groups) {
    __shared__ float scratch[ROW_WARPS];
    pdl_trigger();
    const int warp = threadIdx.x >> 5, at = (threadIdx.x & 31) + 32 * (warp % WPG);
    constexpr int STEP = 32 * WPG;
    const long long task = (long long)blockIdx.x * (ROW_WARPS / WPG) + warp / WPG;
    const int r = (int)(task / groups), g = (int)(task - (long long)r * groups), gw = width / groups, n4 = gw / 4;
    const float4* wg = reinterpret_cast<const float4*>(w + (size_t)g * gw);
    float4 ww[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) if (at + STEP * i < n4) ww[i] = __ldg(wg + at + STEP * i);
    pdl_wait();
    const bool live = r < n_rows;
    const float4* xr = reinterpret_cast<const float4*>(x + (size_t)(live ? (rows ? rows[r] : r) : 0) * width + (size_t)g * gw);
    float4 v[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) v[i] = live && at + STEP * i < n4 ? xr[at + STEP * i] : make_float4(0.f, 0.f, 0.f, 0.f);
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    const float scale = 1.0f / sqrtf(rows_team_sum<WPG>(ss, scratch) / (float)gw + eps);
    if (!live) return;
    TOut* o = out + (size_t)r * width + (size_t)g * gw;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        if (at + STEP * i < n4) {
            const float y[4] = {v[i].x * scale * ww[i].x, v[i].y * scale * ww[i].y, v[i].z * scale * ww[i].z, v[i].w * scale * ww[i].w};
            Vec<TOut, 4>::put(o + 4 * (at + STEP * i), y);
        }
    }
}

template <typename TOut, int NV, int WPG>
__global__ void __launch_bounds__(ROW_WARPS * 32)
group_norm_add_rows_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ ybias,
                           const float* __restrict__ wb, float eps_b, const float* __restrict__ wn, float eps_n,
                           TOut* __restrict__ out, int n_rows, int width, int groups) {
    __shared__ float scratch[2][ROW_WARPS];
    pdl_trigger();
    const int warp = threadIdx.x >> 5, at = (threadIdx.x & 31) + 32 * (warp % WPG);
    constexpr int STEP = 32 * WPG;
    const long long task = (long long)blockIdx.x * (ROW_WARPS / WPG) + warp / WPG;
    const int r = (int)(task / groups), g = (int)(task - (long long)r * groups), gw = width / groups, n4 = gw / 4;
    const size_t col = (size_t)g * gw;
    pdl_wait();
    const bool live = r < n_rows;
    const size_t row = (size_t)(live ? r : 0) * width + col;
    const float4* yr = reinterpret_cast<const float4*>(y + row);
    float4* xr = reinterpret_cast<float4*>(x + row);
    float4 v[NV], xv[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) v[i] = live && at + STEP * i < n4 ? yr[at + STEP * i] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NV; ++i) xv[i] = live && at + STEP * i < n4 ? xr[at + STEP * i] : make_float4(0.f, 0.f, 0.f, 0.f);
    if (ybias) {
        const float4* b = reinterpret_cast<const float4*>(ybias + col);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            if (at + STEP * i < n4) {
                const float4 t = __ldg(b + at + STEP * i);
                v[i].x += t.x; v[i].y += t.y; v[i].z += t.z; v[i].w += t.w;
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    const float scale = 1.0f / sqrtf(rows_team_sum<WPG>(ss, scratch[0]) / (float)gw + eps_b);
    float ss2 = 0.f;
    const float4* b4 = reinterpret_cast<const float4*>(wb + col);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        if (live && at + STEP * i < n4) {
            const float4 t = __ldg(b4 + at + STEP * i);
            xv[i].x += v[i].x * scale * t.x; xv[i].y += v[i].y * scale * t.y; xv[i].z += v[i].z * scale * t.z; xv[i].w += v[i].w * scale * t.w;
            xr[at + STEP * i] = xv[i];
            ss2 += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
        }
    }
    if (out == nullptr) return;
    const float nscale = 1.0f / sqrtf(rows_team_sum<WPG>(ss2, scratch[1]) / (float)gw + eps_n);
    if (!live) return;
    const float4* n4w = reinterpret_cast<const float4*>(wn + col);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        if (at + STEP * i < n4) {
            const float4 t = __ldg(n4w + at + STEP * i);
            const float o[4] = {xv[i].x * nscale * t.x, xv[i].y * nscale * t.y, xv[i].z * nscale * t.z, xv[i].w * nscale * t.w};
            Vec<TOut, 4>::put(out + row + 4 * (at + STEP * i), o);
        }
    }
}

// warps of a block and warps per group: as many warps as keep a thread at REGS vectors of its group or fewer, up to 8
static void plan(int width, int groups, int v, int* warps, int* wpg) {
    int nw = (width + 32 * v * 2 - 1) / (32 * v * 2);         // about two vectors per thread
    nw = nw < 1 ? 1 : (nw > 8 ? 8 : nw);
    int per = groups >= nw ? 1 : nw / groups;
    *wpg = per;
    *warps = groups >= nw ? nw : per * groups;
}

}  // namespace gn
}  // namespace imparo

using namespace imparo;

// out [n_rows, width] = the grouped norm of x's rows (rows[r], or r when rows is null) times w.  groups divides width.
extern "C" int imparo_group_rmsnorm(const float* x, const int* rows, const float* w, float eps, void* out, int out_dtype,
                                    int n_rows, int width, int groups, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (groups < 1 || width < 1 || width % groups != 0) return -2;
    const bool vec = (width / groups) % 4 == 0 && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
    if (vec && n_rows >= gn::MANY_ROWS && width / groups <= 4096) {
        const int nv = (width / groups + 127) / 128, wpg = nv <= 8 ? 1 : (nv <= 16 ? 2 : 4), per = gn::ROW_WARPS / wpg;
        const dim3 grid((unsigned)(((long long)n_rows * groups + per - 1) / per)), block(gn::ROW_WARPS * 32);
#define IMPARO_GR(T_, N_, W_) launch(gn::group_rmsnorm_rows_kernel<T_, N_, W_>, grid, block, 0, stream, x, rows, w, eps, (T_*)out, n_rows, width, groups)
#define IMPARO_GRN(T_) do { if (nv <= 1) IMPARO_GR(T_, 1, 1); else if (nv <= 2) IMPARO_GR(T_, 2, 1); else if (nv <= 4) IMPARO_GR(T_, 4, 1); \
        else if (wpg == 1) IMPARO_GR(T_, 8, 1); else if (wpg == 2) IMPARO_GR(T_, 8, 2); else IMPARO_GR(T_, 8, 4); } while (0)
        if (out_dtype == IMPARO_DT_F32) IMPARO_GRN(float);
        else if (out_dtype == IMPARO_DT_BF16) IMPARO_GRN(__nv_bfloat16);
        else return -1;
#undef IMPARO_GRN
#undef IMPARO_GR
        IMPARO_CHECK_LAUNCH();
        return 0;
    }
    int nw, wpg;
    gn::plan(width, groups, vec ? 4 : 1, &nw, &wpg);
#define IMPARO_GN(T_, V_) launch(gn::group_rmsnorm_kernel<T_, V_>, dim3(n_rows), dim3(32 * nw), 0, stream, x, rows, w, eps, (T_*)out, \
        width, groups, wpg)
    if (out_dtype == IMPARO_DT_F32) { if (vec) IMPARO_GN(float, 4); else IMPARO_GN(float, 1); }
    else if (out_dtype == IMPARO_DT_BF16) { if (vec) IMPARO_GN(__nv_bfloat16, 4); else IMPARO_GN(__nv_bfloat16, 1); }
    else return -1;
#undef IMPARO_GN
    IMPARO_CHECK_LAUNCH();
    return 0;
}

// x float32 [n_rows, width] += the grouped norm of (ybias + y's partials) times wb; y: `parts` tensors [n_rows, width],
// part_stride floats apart, summed in order; ybias float32 [width] or null.  out (or null): [n_rows, width] in out_dtype, the
// grouped norm of the updated rows times wn.
extern "C" int imparo_group_norm_add(float* x, const float* y, int parts, long long part_stride, const float* ybias,
                                     const float* wb, float eps_b, const float* wn, float eps_n, void* out, int out_dtype,
                                     int n_rows, int width, int groups, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (groups < 1 || width < 1 || width % groups != 0 || parts < 1) return -2;
    if (out != nullptr && wn == nullptr) return -2;
    const uintptr_t all = (uintptr_t)x | (uintptr_t)y | (uintptr_t)ybias | (uintptr_t)wb | (uintptr_t)wn | (uintptr_t)out;
    const bool vec = (width / groups) % 4 == 0 && (all & 15) == 0 && (parts == 1 || part_stride % 4 == 0);
    if (vec && parts == 1 && n_rows >= gn::MANY_ROWS && width / groups <= 4096) {
        const int nv = (width / groups + 127) / 128, wpg = nv <= 8 ? 1 : (nv <= 16 ? 2 : 4), per = gn::ROW_WARPS / wpg;
        const dim3 grid((unsigned)(((long long)n_rows * groups + per - 1) / per)), block(gn::ROW_WARPS * 32);
#define IMPARO_GR(T_, N_, W_) launch(gn::group_norm_add_rows_kernel<T_, N_, W_>, grid, block, 0, stream, x, y, ybias, wb, eps_b, wn, eps_n, (T_*)out, \
        n_rows, width, groups)
#define IMPARO_GRN(T_) do { if (nv <= 1) IMPARO_GR(T_, 1, 1); else if (nv <= 2) IMPARO_GR(T_, 2, 1); else if (nv <= 4) IMPARO_GR(T_, 4, 1); \
        else if (wpg == 1) IMPARO_GR(T_, 8, 1); else if (wpg == 2) IMPARO_GR(T_, 8, 2); else IMPARO_GR(T_, 8, 4); } while (0)
        if (out == nullptr || out_dtype == IMPARO_DT_F32) IMPARO_GRN(float);
        else if (out_dtype == IMPARO_DT_BF16) IMPARO_GRN(__nv_bfloat16);
        else return -1;
#undef IMPARO_GRN
#undef IMPARO_GR
        IMPARO_CHECK_LAUNCH();
        return 0;
    }
    int nw, wpg;
    gn::plan(width, groups, vec ? 4 : 1, &nw, &wpg);
#define IMPARO_GN(T_, V_) launch(gn::group_norm_add_kernel<T_, V_>, dim3(n_rows), dim3(32 * nw), 0, stream, x, y, parts, \
        (size_t)part_stride, ybias, wb, eps_b, wn, eps_n, (T_*)out, width, groups, wpg)
    if (out == nullptr || out_dtype == IMPARO_DT_F32) { if (vec) IMPARO_GN(float, 4); else IMPARO_GN(float, 1); }
    else if (out_dtype == IMPARO_DT_BF16) { if (vec) IMPARO_GN(__nv_bfloat16, 4); else IMPARO_GN(__nv_bfloat16, 1); }
    else return -1;
#undef IMPARO_GN
    IMPARO_CHECK_LAUNCH();
    return 0;
}
