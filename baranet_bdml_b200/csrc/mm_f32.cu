// fp32 matrix product in the reference's own arithmetic order: one FMA chain per output, k ascending (reference:
// src/ops/op_mm_optimized.cuh:35-62).
#include "common.cuh"
#include "hybrid.cuh"

namespace bn {

// ---------------------------------------------------------------------------
// GEMM: 64x64 output tile, 256 threads, 4x4 outputs per thread, k in slabs of 16
// ---------------------------------------------------------------------------
constexpr int MM_T = 64;
constexpr int MM_K = 16;

__global__ void __launch_bounds__(256)
mm_f32_kernel(const float* __restrict__ A, int64_t a_rs, int64_t a_cs, const float* __restrict__ B, int64_t b_rs,
              int64_t b_cs, float* __restrict__ C, int64_t c_rs, int64_t c_cs, int M, int K, int N) {
    __shared__ float As[MM_K][MM_T + 4];
    __shared__ float Bs[MM_K][MM_T + 4];
    const int tid = threadIdx.x;
    const int tx = tid % 16, ty = tid / 16;
    const int row0 = blockIdx.y * MM_T, col0 = blockIdx.x * MM_T;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;

    for (int k0 = 0; k0 < K; k0 += MM_K) {
        // stage A (64 rows x 16 k) and B (16 k x 64 cols); out-of-range -> 0
#pragma unroll
        for (int e = tid; e < MM_T * MM_K; e += 256) {
            int kk = e % MM_K, r = e / MM_K;
            int gr = row0 + r, gk = k0 + kk;
            As[kk][r] = (gr < M && gk < K) ? A[gr * a_rs + gk * a_cs] : 0.0f;
        }
#pragma unroll
        for (int e = tid; e < MM_T * MM_K; e += 256) {
            int c = e % MM_T, kk = e / MM_T;
            int gc = col0 + c, gk = k0 + kk;
            Bs[kk][c] = (gc < N && gk < K) ? B[gk * b_rs + gc * b_cs] : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < MM_K; ++kk) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = As[kk][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = Bs[kk][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        int gr = row0 + ty * 4 + i;
        if (gr >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            int gc = col0 + tx * 4 + j;
            if (gc < N) C[gr * c_rs + gc * c_cs] = acc[i][j];
        }
    }
}

// x = act(x + bias) in place, fp32 rows (the unfused form of the products with a bias or an activation)
__global__ void __launch_bounds__(256)
bias_act_kernel(float* x, int64_t ld, const float* bias, long long n, int cols, int act) {
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) {
        const int64_t r = i / cols, c = i - r * cols;
        x[r * ld + c] = activation_exact(act, x[r * ld + c] + (bias ? bias[c] : 0.f));
    }
}

}  // namespace bn

using namespace bn;

extern "C" int bn_mm_f32(const float* A, int64_t a_rs, int64_t a_cs, const float* B, int64_t b_rs, int64_t b_cs,
                         float* C, int64_t c_rs, int64_t c_cs, int M, int K, int N, bn_stream_t stream) {
    if (!A || !B || !C) return fail(BN_ERR_INVALID_ARG, "bn_mm_f32: null pointer");
    if (M < 0 || K < 0 || N < 0) return fail(BN_ERR_INVALID_ARG, "bn_mm_f32: negative size");
    if (int rc = require_sm100()) return rc;
    if (M == 0 || N == 0) return BN_OK;
    dim3 grid(ceil_div(N, MM_T), ceil_div(M, MM_T));
    if (grid.y > 65535) return fail(BN_ERR_UNSUPPORTED, "bn_mm_f32: M=%d too large", M);
    mm_f32_kernel<<<grid, 256, 0, as_stream(stream)>>>(A, a_rs, a_cs, B, b_rs, b_cs, C, c_rs, c_cs, M, K, N);
    return launch_status("bn_mm_f32");
}

extern "C" int bn_bias_act_f32(float* x, int64_t ld, const float* bias, int rows, int cols, int act, bn_stream_t stream) {
    if (!x) return fail(BN_ERR_INVALID_ARG, "bn_bias_act_f32: null pointer");
    if (rows < 0 || cols < 0 || act < 0 || act > BN_ACT_LAST) return fail(BN_ERR_INVALID_ARG, "bn_bias_act_f32: bad shape or activation");
    if (int rc = require_sm100()) return rc;
    const long long n = (long long)rows * cols;
    if (n == 0) return BN_OK;
    const long long blocks = (n + 255) / 256;
    bias_act_kernel<<<(unsigned)(blocks < 4096 ? blocks : 4096), 256, 0, as_stream(stream)>>>(x, ld, bias, n, cols, act);
    return launch_status("bn_bias_act_f32");
}
