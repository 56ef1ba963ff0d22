// The fp32 residual stream of the pre-norm models and everything that happens to it between two products, one launch
// each: add a sublayer's output (optionally RMS-normed with a weight of its own first), add a constant row vector, keep
// the fp32 sum, emit it rounded for a product that reads the stream itself, and emit its layer norm or RMS norm.
//
//   d    = delta                                   or  delta / sqrt(mean(delta^2) + delta_eps) * delta_w
//   x'   = x + d + row                             (each of the three optional)
//   cast = round(x')                               optionally followed, lo_offset columns on, by round(x' - round(x'))
//   y    = (x' - mean) / sqrt(var + eps) * w + b   (center)   or   x' / sqrt(mean(x'^2) + eps) * w
//
// HBM-bound.  A row stays in registers between the passes (hidden <= 4096, rows in 16-byte pieces); other shapes keep it
// in shared memory.  The variance is the mean of the squared deviations, taken in a second pass over the registers.
#include "common.cuh"
#include "hybrid.cuh"

namespace bn {

struct ResidualNormParams {
    const float* x;
    const void* delta;
    const float* delta_w;
    const float* row;
    float* x_out;
    void* cast;
    const float *w, *b;
    void* y;
    int64_t delta_ld, cast_ld, y_ld;
    int rows, hidden, lo_offset, center;
    float delta_eps, eps;
};

constexpr int RS_THREADS = 256;

// NV = float4 pieces per thread: hidden <= 1024 * NV, hidden % 4 == 0, every row start 16-byte (T = bf16: 8-byte) aligned
template <typename T, typename TD, int NV>
__global__ void __launch_bounds__(RS_THREADS)
residual_norm_regs_kernel(const ResidualNormParams p) {
    __shared__ float sh[RS_THREADS / 32];
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int pieces = p.hidden / 4;
    const float inv_n = 1.f / (float)p.hidden;
    for (int r = blockIdx.x; r < p.rows; r += gridDim.x) {
        float v[NV][4];
#pragma unroll
        for (int k = 0; k < NV; ++k) v[k][0] = v[k][1] = v[k][2] = v[k][3] = 0.f;
        if (p.delta) {
            const TD* dr = static_cast<const TD*>(p.delta) + (int64_t)r * p.delta_ld;
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int c = threadIdx.x + k * RS_THREADS;
                if (c < pieces) load4(dr + 4 * c, v[k]);
            }
        }
        float xv[NV][4];
        if (p.x) {
            const float* xr = p.x + (int64_t)r * p.hidden;
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int c = threadIdx.x + k * RS_THREADS;
                if (c < pieces) load4(xr + 4 * c, xv[k]);
            }
        }
        if (p.delta_w) {
            float s = 0.f;
#pragma unroll
            for (int k = 0; k < NV; ++k)
#pragma unroll
                for (int e = 0; e < 4; ++e) s = fmaf(v[k][e], v[k][e], s);
            const float inv = rsqrtf(block_sum<RS_THREADS>(s, sh) * inv_n + p.delta_eps);
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int c = threadIdx.x + k * RS_THREADS;
                if (c < pieces) {
                    float w4[4];
                    load4(p.delta_w + 4 * c, w4);
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[k][e] = v[k][e] * inv * w4[e];
                }
            }
        }
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * RS_THREADS;
            if (c < pieces) {
                if (p.x) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[k][e] += xv[k][e];
                }
                if (p.row) {
                    float w4[4];
                    load4(p.row + 4 * c, w4);
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[k][e] += w4[e];
                }
                if (p.x_out) store4(p.x_out + (int64_t)r * p.hidden + 4 * c, v[k]);
                if (p.cast) {
                    T* cr = static_cast<T*>(p.cast) + (int64_t)r * p.cast_ld + 4 * c;
                    store4(cr, v[k]);
                    if (p.lo_offset) {
                        float lo[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e) lo[e] = v[k][e] - round_to<T>(v[k][e]);
                        store4(cr + p.lo_offset, lo);
                    }
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) s += p.center ? v[k][e] : v[k][e] * v[k][e];
            }
        }
        if (!p.w) continue;
        s = block_sum<RS_THREADS>(s, sh) * inv_n;
        float mean = 0.f;
        if (p.center) {
            mean = s;
            float q = 0.f;
#pragma unroll
            for (int k = 0; k < NV; ++k)
                if (threadIdx.x + k * RS_THREADS < pieces) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) q = fmaf(v[k][e] - mean, v[k][e] - mean, q);
                }
            s = block_sum<RS_THREADS>(q, sh) * inv_n;
        }
        const float inv = rsqrtf(s + p.eps);
        T* yr = static_cast<T*>(p.y) + (int64_t)r * p.y_ld;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * RS_THREADS;
            if (c < pieces) {
                float w4[4], b4[4] = {0.f, 0.f, 0.f, 0.f}, o4[4];
                load4(p.w + 4 * c, w4);
                if (p.b) load4(p.b + 4 * c, b4);
#pragma unroll
                for (int e = 0; e < 4; ++e) o4[e] = fmaf((v[k][e] - mean) * inv, w4[e], b4[e]);
                store4(yr + 4 * c, o4);
            }
        }
    }
}

// any hidden and any strides; the row is kept in shared memory
template <typename T, typename TD>
__global__ void __launch_bounds__(RS_THREADS)
residual_norm_any_kernel(const ResidualNormParams p) {
    extern __shared__ float row_buf[];
    __shared__ float sh[RS_THREADS / 32];
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const float n = (float)p.hidden;
    for (int r = blockIdx.x; r < p.rows; r += gridDim.x) {
        const TD* dr = p.delta ? static_cast<const TD*>(p.delta) + (int64_t)r * p.delta_ld : nullptr;
        float inv_d = 1.f;
        if (dr && p.delta_w) {
            float s = 0.f;
            for (int i = threadIdx.x; i < p.hidden; i += RS_THREADS) { const float d = to_f(dr[i]); s = fmaf(d, d, s); }
            inv_d = rsqrtf(block_sum<RS_THREADS>(s, sh) / n + p.delta_eps);
        }
        float s = 0.f;
        for (int i = threadIdx.x; i < p.hidden; i += RS_THREADS) {
            float v = dr ? to_f(dr[i]) : 0.f;
            if (dr && p.delta_w) v = v * inv_d * p.delta_w[i];
            if (p.x) v += p.x[(int64_t)r * p.hidden + i];
            if (p.row) v += p.row[i];
            row_buf[i] = v;               // read back by the same thread only
            if (p.x_out) p.x_out[(int64_t)r * p.hidden + i] = v;
            if (p.cast) {
                T* cr = static_cast<T*>(p.cast) + (int64_t)r * p.cast_ld + i;
                *cr = from_f<T>(v);
                if (p.lo_offset) cr[p.lo_offset] = from_f<T>(v - round_to<T>(v));
            }
            s += p.center ? v : v * v;
        }
        if (!p.w) continue;
        s = block_sum<RS_THREADS>(s, sh) / n;
        float mean = 0.f;
        if (p.center) {
            mean = s;
            float q = 0.f;
            for (int i = threadIdx.x; i < p.hidden; i += RS_THREADS) q = fmaf(row_buf[i] - mean, row_buf[i] - mean, q);
            s = block_sum<RS_THREADS>(q, sh) / n;
        }
        const float inv = rsqrtf(s + p.eps);
        T* yr = static_cast<T*>(p.y) + (int64_t)r * p.y_ld;
        for (int i = threadIdx.x; i < p.hidden; i += RS_THREADS)
            yr[i] = from_f<T>(fmaf((row_buf[i] - mean) * inv, p.w[i], p.b ? p.b[i] : 0.f));
    }
}

template <typename T, typename TD>
static int residual_norm_launch(const ResidualNormParams& p, bn_stream_t stream) {
    const char* what = "bn_residual_norm";
    int dev = 0, sms = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const long long cap = (long long)sms * 8;
    const unsigned grid = (unsigned)(p.rows < cap ? p.rows : cap);
    const uintptr_t f32s = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.delta_w) |
                           reinterpret_cast<uintptr_t>(p.row) | reinterpret_cast<uintptr_t>(p.x_out) |
                           reinterpret_cast<uintptr_t>(p.w) | reinterpret_cast<uintptr_t>(p.b);
    const uintptr_t others = reinterpret_cast<uintptr_t>(p.delta) | reinterpret_cast<uintptr_t>(p.cast) |
                             reinterpret_cast<uintptr_t>(p.y);
    const bool vec = p.hidden % 4 == 0 && p.hidden <= 4096 && p.delta_ld % 4 == 0 && p.cast_ld % 4 == 0 && p.y_ld % 4 == 0 &&
                     p.lo_offset % 4 == 0 && ((f32s | others) & 15) == 0;
    cudaStream_t st = as_stream(stream);
    if (vec && p.hidden <= 1024) launch_dependent(residual_norm_regs_kernel<T, TD, 1>, grid, RS_THREADS, 0, st, p);
    else if (vec && p.hidden <= 2048) launch_dependent(residual_norm_regs_kernel<T, TD, 2>, grid, RS_THREADS, 0, st, p);
    else if (vec) launch_dependent(residual_norm_regs_kernel<T, TD, 4>, grid, RS_THREADS, 0, st, p);
    else {
        const size_t smem = (size_t)p.hidden * sizeof(float);
        if (smem > 200 * 1024) return fail(BN_ERR_UNSUPPORTED, "%s: hidden=%d (at most 51200)", what, p.hidden);
        if (smem > 48 * 1024) {
            cudaError_t e = cudaFuncSetAttribute(residual_norm_any_kernel<T, TD>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 (int)smem);
            if (e != cudaSuccess) return fail(BN_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
        }
        launch_dependent(residual_norm_any_kernel<T, TD>, grid, RS_THREADS, smem, st, p);
    }
    return launch_status(what);
}

// out = act(a) * b, fp32 rows (the unfused form of the gated products)
__global__ void __launch_bounds__(256)
act_mul_kernel(const float* a, int64_t a_ld, const float* b, int64_t b_ld, float* out, int64_t out_ld, long long n, int cols,
               int act) {
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) {
        const int64_t r = i / cols, c = i - r * cols;
        out[r * out_ld + c] = activation_exact(act, a[r * a_ld + c]) * b[r * b_ld + c];
    }
}

}  // namespace bn

using namespace bn;

extern "C" int bn_residual_norm(const float* x, const void* delta, int64_t delta_ld, int delta_dtype, const float* delta_w,
                                float delta_eps, const float* row, float* x_out, void* cast, int64_t cast_ld, int lo_offset,
                                const float* w, const float* b, void* y, int64_t y_ld, int center, int dtype, int rows,
                                int hidden, float eps, bn_stream_t stream) {
    const char* what = "bn_residual_norm";
    if (!x && !delta) return fail(BN_ERR_INVALID_ARG, "%s: neither a stream nor a delta", what);
    if ((w && !y) || (!w && !x_out && !cast)) return fail(BN_ERR_INVALID_ARG, "%s: nothing to write", what);
    if (rows < 0 || hidden <= 0 || lo_offset < 0) return fail(BN_ERR_INVALID_ARG, "%s: bad shape rows=%d hidden=%d", what, rows, hidden);
    if ((dtype | delta_dtype) & ~1) return fail(BN_ERR_INVALID_ARG, "%s: dtype %d / %d", what, dtype, delta_dtype);
    if (int rc = require_sm100()) return rc;
    if (rows == 0) return BN_OK;
    ResidualNormParams p{x, delta, delta_w, row, x_out, cast, w, b, y, delta_ld, cast_ld, y_ld, rows, hidden, lo_offset, center,
                         delta_eps, eps};
    if (dtype == 0 && delta_dtype == 0) return residual_norm_launch<float, float>(p, stream);
    if (dtype == 0) return fail(BN_ERR_UNSUPPORTED, "%s: a bf16 delta on the fp32 path", what);
    if (delta_dtype == 0) return residual_norm_launch<__nv_bfloat16, float>(p, stream);
    return residual_norm_launch<__nv_bfloat16, __nv_bfloat16>(p, stream);
}

extern "C" int bn_act_mul_f32(const float* a, int64_t a_ld, const float* b, int64_t b_ld, float* out, int64_t out_ld, int rows,
                              int cols, int act, bn_stream_t stream) {
    if (!a || !b || !out) return fail(BN_ERR_INVALID_ARG, "bn_act_mul_f32: null pointer");
    if (rows < 0 || cols < 0 || act < 0 || act > BN_ACT_LAST) return fail(BN_ERR_INVALID_ARG, "bn_act_mul_f32: bad shape or activation");
    if (int rc = require_sm100()) return rc;
    const long long n = (long long)rows * cols;
    if (n == 0) return BN_OK;
    const long long blocks = (n + 255) / 256;
    act_mul_kernel<<<(unsigned)(blocks < 4096 ? blocks : 4096), 256, 0, as_stream(stream)>>>(a, a_ld, b, b_ld, out, out_ld, n,
                                                                                       cols, act);
    return launch_status("bn_act_mul_f32");
}
