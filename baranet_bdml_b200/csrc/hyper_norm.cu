// A residual stream kept as several fp32 copies ("streams") that a sublayer reads and writes through small matrices, and
// everything that happens to them between two products, in one launch:
//
//   x'_t = sum_s mix[s][t] x_s + w_out[t] * (delta * delta_scale)     delta: the output of the sublayer before, optional
//   u    = sum_t w_in[t] x'_t
//   y    = u / sqrt(mean(u^2) + eps) * w                              what the next sublayer's product reads
//
// n_in old streams become n_out new ones.  The matrix need not be square: the first sublayer of a model finds ONE stream (the
// embedding, of which all streams are copies), and where the new streams themselves are not wanted the caller folds w_in
// into mix and w_out and asks for one.  Stream s of row r starts at x + (r * n_in + s) * hidden.
//
// HBM-bound.  The coefficients travel with the launch (constant bank); a row's pieces stay in registers between the mixing
// and the norm (hidden <= 4096, at most 4 streams, bf16), other shapes keep u in shared memory.
#include "common.cuh"
#include "hybrid.cuh"

namespace bn {

constexpr int HY_THREADS = 256, HY_MAX = 16;

struct HyperParams {
    const float* x;
    const void* delta;
    const float* delta_scale;      // (hidden) or null
    float* x_out;                  // or null
    const float* w;                // null: y is not wanted
    void* y;
    int64_t delta_ld, y_ld;
    int rows, hidden, n_in, n_out;
    float eps;
    float mix[HY_MAX * HY_MAX], w_out[HY_MAX], w_in[HY_MAX];       // mix[s * n_out + t]
};

// NV = float4 pieces per thread: hidden <= 1024 * NV, hidden % 4 == 0, every row start 16-byte (bf16: 8-byte) aligned
template <typename T, int NV, int NI, int NO>
__global__ void __launch_bounds__(HY_THREADS)
hyper_norm_regs_kernel(const __grid_constant__ HyperParams p) {
    __shared__ float sh[HY_THREADS / 32];
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int pieces = p.hidden / 4;
    const float inv_n = 1.f / (float)p.hidden;
    for (int r = blockIdx.x; r < p.rows; r += gridDim.x) {
        float xv[NV][NI][4], d[NV][4];
        const float* xr = p.x + (int64_t)r * NI * p.hidden;
        const T* dr = static_cast<const T*>(p.delta) + (int64_t)r * p.delta_ld;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * HY_THREADS;
            d[k][0] = d[k][1] = d[k][2] = d[k][3] = 0.f;
#pragma unroll
            for (int s = 0; s < NI; ++s) xv[k][s][0] = xv[k][s][1] = xv[k][s][2] = xv[k][s][3] = 0.f;
            if (c < pieces) {
#pragma unroll
                for (int s = 0; s < NI; ++s) load4(xr + (int64_t)s * p.hidden + 4 * c, xv[k][s]);
                if (p.delta) load4(dr + 4 * c, d[k]);
            }
        }
        float u[NV][4], ss = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * HY_THREADS;
            if (p.delta_scale && c < pieces) {
                float w4[4];
                load4(p.delta_scale + 4 * c, w4);
#pragma unroll
                for (int e = 0; e < 4; ++e) d[k][e] *= w4[e];
            }
            u[k][0] = u[k][1] = u[k][2] = u[k][3] = 0.f;
#pragma unroll
            for (int t = 0; t < NO; ++t) {
                float n4[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    n4[e] = p.w_out[t] * d[k][e];
#pragma unroll
                    for (int s = 0; s < NI; ++s) n4[e] = fmaf(p.mix[s * NO + t], xv[k][s][e], n4[e]);
                    u[k][e] = fmaf(p.w_in[t], n4[e], u[k][e]);
                }
                if (p.x_out && c < pieces) store4(p.x_out + ((int64_t)r * NO + t) * p.hidden + 4 * c, n4);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) ss = fmaf(u[k][e], u[k][e], ss);
        }
        if (!p.w) continue;
        const float inv = rsqrtf(block_sum<HY_THREADS>(ss, sh) * inv_n + p.eps);
        T* yr = static_cast<T*>(p.y) + (int64_t)r * p.y_ld;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * HY_THREADS;
            if (c < pieces) {
                float w4[4], o4[4];
                load4(p.w + 4 * c, w4);
#pragma unroll
                for (int e = 0; e < 4; ++e) o4[e] = u[k][e] * inv * w4[e];
                store4(yr + 4 * c, o4);
            }
        }
    }
}

// any hidden, any number of streams up to HY_MAX, any strides
template <typename T>
__global__ void __launch_bounds__(HY_THREADS)
hyper_norm_any_kernel(const __grid_constant__ HyperParams p) {
    extern __shared__ float row_buf[];
    __shared__ float sh[HY_THREADS / 32], s_mix[HY_MAX * HY_MAX], s_out[HY_MAX], s_in[HY_MAX];
    for (int i = threadIdx.x; i < p.n_in * p.n_out; i += HY_THREADS) s_mix[i] = p.mix[i];
    if (threadIdx.x < p.n_out) { s_out[threadIdx.x] = p.w_out[threadIdx.x]; s_in[threadIdx.x] = p.w_in[threadIdx.x]; }
    __syncthreads();
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    for (int r = blockIdx.x; r < p.rows; r += gridDim.x) {
        const T* dr = p.delta ? static_cast<const T*>(p.delta) + (int64_t)r * p.delta_ld : nullptr;
        float ss = 0.f;
        for (int i = threadIdx.x; i < p.hidden; i += HY_THREADS) {
            float d = dr ? to_f(dr[i]) : 0.f;
            if (p.delta_scale) d *= p.delta_scale[i];
            float u = 0.f;
            for (int t = 0; t < p.n_out; ++t) {
                float n = s_out[t] * d;
                for (int s = 0; s < p.n_in; ++s) n = fmaf(s_mix[s * p.n_out + t], p.x[((int64_t)r * p.n_in + s) * p.hidden + i], n);
                if (p.x_out) p.x_out[((int64_t)r * p.n_out + t) * p.hidden + i] = n;
                u = fmaf(s_in[t], n, u);
            }
            row_buf[i] = u;               // read back by the same thread only
            ss = fmaf(u, u, ss);
        }
        if (!p.w) continue;
        const float inv = rsqrtf(block_sum<HY_THREADS>(ss, sh) / (float)p.hidden + p.eps);
        T* yr = static_cast<T*>(p.y) + (int64_t)r * p.y_ld;
        for (int i = threadIdx.x; i < p.hidden; i += HY_THREADS) yr[i] = from_f<T>(row_buf[i] * inv * p.w[i]);
    }
}

template <int NV, int NI, int NO>
static void hyper_launch(unsigned grid, cudaStream_t st, const HyperParams& p) {
    launch_dependent(hyper_norm_regs_kernel<__nv_bfloat16, NV, NI, NO>, grid, HY_THREADS, 0, st, p);
}

// the stream counts that have a register form; false: none
template <int NV>
static bool hyper_regs(unsigned grid, cudaStream_t st, const HyperParams& p) {
    switch (p.n_in * 8 + p.n_out) {
        case 1 * 8 + 1: hyper_launch<NV, 1, 1>(grid, st, p); return true;
        case 1 * 8 + 2: hyper_launch<NV, 1, 2>(grid, st, p); return true;
        case 1 * 8 + 3: hyper_launch<NV, 1, 3>(grid, st, p); return true;
        case 1 * 8 + 4: hyper_launch<NV, 1, 4>(grid, st, p); return true;
        case 2 * 8 + 1: hyper_launch<NV, 2, 1>(grid, st, p); return true;
        case 2 * 8 + 2: hyper_launch<NV, 2, 2>(grid, st, p); return true;
        case 3 * 8 + 1: hyper_launch<NV, 3, 1>(grid, st, p); return true;
        case 3 * 8 + 3: hyper_launch<NV, 3, 3>(grid, st, p); return true;
        case 4 * 8 + 1: hyper_launch<NV, 4, 1>(grid, st, p); return true;
        case 4 * 8 + 4: hyper_launch<NV, 4, 4>(grid, st, p); return true;
    }
    return false;
}

template <typename T>
static int hyper_any(unsigned grid, cudaStream_t st, const HyperParams& p) {
    const char* what = "bn_hyper_norm";
    const size_t smem = (size_t)p.hidden * sizeof(float);
    if (smem > 200 * 1024) return fail(BN_ERR_UNSUPPORTED, "%s: hidden=%d (at most 51200)", what, p.hidden);
    if (smem > 40 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(hyper_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail(BN_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
    }
    launch_dependent(hyper_norm_any_kernel<T>, grid, HY_THREADS, smem, st, p);
    return launch_status(what);
}

}  // namespace bn

using namespace bn;

extern "C" int bn_hyper_norm(const float* x, int n_in, int n_out, const float* mix, const float* w_out, const float* w_in,
                             const void* delta, int64_t delta_ld, const float* delta_scale, float* x_out, const float* w, void* y,
                             int64_t y_ld, int dtype, int rows, int hidden, float eps, bn_stream_t stream) {
    const char* what = "bn_hyper_norm";
    if (!x || !mix || !w_out || !w_in) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if ((w && !y) || (!w && !x_out)) return fail(BN_ERR_INVALID_ARG, "%s: nothing to write", what);
    if (rows < 0 || hidden <= 0 || n_in <= 0 || n_out <= 0 || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape rows=%d hidden=%d streams %d -> %d", what, rows, hidden, n_in, n_out);
    if (n_in > HY_MAX || n_out > HY_MAX) return fail(BN_ERR_UNSUPPORTED, "%s: %d -> %d streams (at most %d)", what, n_in, n_out, HY_MAX);
    if (int rc = require_sm100()) return rc;
    if (rows == 0) return BN_OK;
    HyperParams p{};
    p.x = x; p.delta = delta; p.delta_scale = delta_scale; p.x_out = x_out; p.w = w; p.y = y;
    p.delta_ld = delta_ld; p.y_ld = y_ld; p.rows = rows; p.hidden = hidden; p.n_in = n_in; p.n_out = n_out; p.eps = eps;
    for (int i = 0; i < n_in * n_out; ++i) p.mix[i] = mix[i];
    for (int t = 0; t < n_out; ++t) { p.w_out[t] = w_out[t]; p.w_in[t] = w_in[t]; }
    int dev = 0, sms = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const long long cap = (long long)sms * 8;
    const unsigned grid = (unsigned)(rows < cap ? rows : cap);
    const uintptr_t all = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(delta) | reinterpret_cast<uintptr_t>(delta_scale) |
                          reinterpret_cast<uintptr_t>(x_out) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(y);
    const bool vec = dtype == 1 && hidden % 4 == 0 && hidden <= 4096 && delta_ld % 4 == 0 && y_ld % 4 == 0 && (all & 15) == 0 &&
                     n_in <= 4 && n_out <= 4;
    cudaStream_t st = as_stream(stream);
    if (vec && hidden <= 1024 && hyper_regs<1>(grid, st, p)) return launch_status(what);
    if (vec && hidden > 1024 && hidden <= 2048 && hyper_regs<2>(grid, st, p)) return launch_status(what);
    if (vec && hidden > 2048 && hyper_regs<4>(grid, st, p)) return launch_status(what);
    return dtype == 0 ? hyper_any<float>(grid, st, p) : hyper_any<__nv_bfloat16>(grid, st, p);
}
