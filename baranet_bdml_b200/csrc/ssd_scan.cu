// The selective state-space recurrence of a prompt portion in chunks of 64 tokens, on warp-level tensor cores: within a
// chunk the recurrence is written out as products (the state-space dual form), between chunks the fp32 state is carried in
// registers.  bn_ssm_scan's fast path (bf16 inputs).
//
// With c_i the running sum of the chunk's log decays (c_i <= 0, falling) and S the state before the chunk (N x P):
//   y_i  = e^{c_i} S^T C_i  +  sum_{j <= i} e^{c_i - c_j} dt_j (C_i . B_j) x_j  +  D x_i
//   S'   = e^{c_last} S     +  sum_j e^{c_last - c_j} dt_j B_j x_j^T
// Decays, step sizes and the state are fp32 quantities that meet bf16 operands in these products.  Each of them goes in as
// TWO bf16 numbers, its rounding and the remainder of that rounding, so a product sees 16 of its bits; x, B and C are
// bf16 already and go in as they are.  Sums are fp32.
//
// CTA = (sequence, head, slice of 16 W values), W warps; warp w owns 16 values: their state as MMA accumulators
// (16 x N fp32), the outputs of all 64 tokens for them.  An accumulator fragment of (value, state) is, register for
// register, the B fragment of (state, value), so S enters S^T C without leaving the registers.  The 64 x 64 matrix of the
// first sum is shared: the warps take its row blocks in turn and leave its two bf16 parts in shared memory, only the blocks
// on and below the diagonal (55 KB and 128 registers a thread: four CTAs per SM).
#include "common.cuh"
#include "hybrid.cuh"
#include "mamba2.cuh"

namespace bn {

using namespace ptx;

constexpr int SD_Q = 64;                       // tokens per chunk
constexpr int SD_MBLOCKS = 10;                 // 16 x 16 blocks on and below the diagonal of the 64 x 64 matrix

// Element offset of row r, columns 8 c .. 8 c + 7 (c = 0, 1) of block (mb, kb): blocks are packed, a row is 32 bytes, and
// rows 4-7 of eight swap their halves, so that eight rows of one half lie in different banks.
__device__ __forceinline__ int sd_m_offset(int mb, int kb, int r, int c) {
    return (mb * (mb + 1) / 2 + kb) * 256 + r * 16 + ((c ^ (r >> 2 & 1)) << 3);
}

__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}

// NP: N rounded up to a multiple of 16 that the kernel is built for; columns N .. NP - 1 are zeros
template <int NP>
__global__ void __launch_bounds__(128, 4)
ssd_scan_kernel(const SsmScanParams p, int slices) {
    constexpr int LDN = NP + 8;                // row stride of the B and C tiles, elements
    extern __shared__ __align__(16) uint8_t smem[];
    const int W = blockDim.x / 32, warp = threadIdx.x / 32, lane = threadIdx.x % 32, g = lane / 4, j = lane % 4;
    const int PW = W * 16, LDX = PW + 8;
    __nv_bfloat16* sB = reinterpret_cast<__nv_bfloat16*>(smem);          // [64][LDN]
    __nv_bfloat16* sC = sB + SD_Q * LDN;                                 // [64][LDN]
    __nv_bfloat16* sMh = sC + SD_Q * LDN;                                // packed blocks, high and low parts
    __nv_bfloat16* sMl = sMh + SD_MBLOCKS * 256;
    __nv_bfloat16* sX = sMl + SD_MBLOCKS * 256;                          // [64][LDX]
    float* s_cum = reinterpret_cast<float*>(sX + SD_Q * LDX);            // [64] c_i
    float* s_dt = s_cum + SD_Q;                                          // [64]
    float* s_w = s_dt + SD_Q;                                            // [64] e^{c_last - c_j} dt_j
    grid_dependency_wait();
    grid_launch_dependents();
    const int slice = blockIdx.x % slices, h = blockIdx.x / slices % p.H, b = blockIdx.x / (slices * p.H);
    const int grp = h / (p.H / p.G), slot = p.seq_ids ? p.seq_ids[b] : b;
    const int v0 = slice * PW, nv = min(PW, p.P - v0);                   // this CTA's values
    const float D = p.D[h];
    const int inner = p.H * p.P;
    const __nv_bfloat16* xbc = static_cast<const __nv_bfloat16*>(p.xbc) + (int64_t)b * p.S * p.xbc_ld;
    const __nv_bfloat16* gx = xbc + h * p.P + v0;
    const __nv_bfloat16* gB = xbc + inner + grp * p.N;
    const __nv_bfloat16* gC = gB + p.G * p.N;
    const uint32_t uB = smem_u32(sB), uC = smem_u32(sC), uMh = smem_u32(sMh), uMl = smem_u32(sMl), uX = smem_u32(sX);

    // state: st[t] = values 16 warp + g (+ 8), state columns 8 t + 2 j (+ 1)
    float st[NP / 8][4];
    float* state = p.state + (((int64_t)slot * p.H + h) * p.P + v0 + warp * 16) * p.N;
#pragma unroll
    for (int t = 0; t < NP / 8; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = g + (e / 2) * 8, n = t * 8 + 2 * j + e % 2;
            st[t][e] = warp * 16 + r < nv && n < p.N ? state[(int64_t)r * p.N + n] : 0.f;
        }

    for (int t0 = 0; t0 < p.S; t0 += SD_Q) {
        const int nt = min(SD_Q, p.S - t0);
        __syncthreads();                       // the chunk before has been read
        // ---- tiles of the chunk (pieces of 8; beyond the sequence or the matrix: zeros)
        for (int i = threadIdx.x; i < SD_Q * (NP / 8); i += blockDim.x) {
            const int r = i / (NP / 8), c = i % (NP / 8) * 8;
            const bool in = r < nt && c < p.N;                           // N is a multiple of 8
            const int64_t o = in ? (int64_t)(t0 + r) * p.xbc_ld + c : 0;
            cp_async_16(uB + (r * LDN + c) * 2, gB + o, in ? 16 : 0);
            cp_async_16(uC + (r * LDN + c) * 2, gC + o, in ? 16 : 0);
        }
        for (int i = threadIdx.x; i < SD_Q * (PW / 8); i += blockDim.x) {
            const int r = i / (PW / 8), c = i % (PW / 8) * 8;
            const bool in = r < nt && c < nv;                            // P is a multiple of 8
            cp_async_16(uX + (r * LDX + c) * 2, gx + (in ? (int64_t)(t0 + r) * p.xbc_ld + c : 0), in ? 16 : 0);
        }
        // the next chunk's values on their way to L2 (its B and C serve all heads of a group and are there already)
        if (threadIdx.x < SD_Q && t0 + SD_Q + (int)threadIdx.x < p.S)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(gx + (int64_t)(t0 + SD_Q + threadIdx.x) * p.xbc_ld));
        if (warp == 0) {                       // running sum of the log decays, two tokens per lane
            const int i0 = 2 * lane;
            const int64_t row = (int64_t)b * p.S + t0;
            float a0 = 0.f, a1 = 0.f, d0 = 0.f, d1 = 0.f;
            if (i0 < nt) { a0 = p.a[(row + i0) * p.H + h]; d0 = p.dt[(row + i0) * p.H + h]; }
            if (i0 + 1 < nt) { a1 = p.a[(row + i0 + 1) * p.H + h]; d1 = p.dt[(row + i0 + 1) * p.H + h]; }
            float s = a0 + a1;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float u = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += u;
            }
            // tokens beyond the sequence add no decay and have step 0, so the last sum is the chunk's whole decay
            const float before = s - (a0 + a1), last = __shfl_sync(0xffffffffu, s, 31);
            s_cum[i0] = before + a0;
            s_cum[i0 + 1] = s;
            s_dt[i0] = d0;
            s_dt[i0 + 1] = d1;
            s_w[i0] = expf(last - (before + a0)) * d0;
            s_w[i0 + 1] = expf(last - s) * d1;
        }
        cp_async_wait_all();
        __syncthreads();
        // ---- M = (C B^T) e^{c_i - c_j} dt_j for j <= i, 16 rows at a time
        for (int mb = warp; mb < SD_Q / 16; mb += W) {
            float acc[SD_Q / 8][4];
#pragma unroll
            for (int t = 0; t < SD_Q / 8; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
            const uint32_t ca = uC + ((mb * 16 + lane % 16) * LDN + (lane / 16) * 8) * 2;
#pragma unroll
            for (int ks = 0; ks < NP / 16; ++ks) {
                uint32_t a0, a1, a2, a3;
                ldmatrix_x4(ca + ks * 32, a0, a1, a2, a3);
#pragma unroll
                for (int t2 = 0; t2 < SD_Q / 16; ++t2) {
                    if (t2 > mb) break;        // columns after the rows
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4(uB + ((t2 * 16 + (lane / 16) * 8 + lane % 8) * LDN + ks * 16 + (lane / 8 % 2) * 8) * 2, b0, b1, b2, b3);
                    mma_bf16_16816(acc[2 * t2], a0, a1, a2, a3, b0, b1);
                    mma_bf16_16816(acc[2 * t2 + 1], a0, a1, a2, a3, b2, b3);
                }
            }
            const int i0 = mb * 16 + g, i1 = i0 + 8;
            const float c0 = s_cum[i0], c1 = s_cum[i1];
#pragma unroll
            for (int t = 0; t < SD_Q / 8; ++t) {
                if (t / 2 > mb) break;
                const int q0 = t * 8 + 2 * j, q1 = q0 + 1;
                const float e0 = s_cum[q0], e1 = s_cum[q1], d0 = s_dt[q0], d1 = s_dt[q1];
                const float m00 = q0 <= i0 ? acc[t][0] * __expf(c0 - e0) * d0 : 0.f, m01 = q1 <= i0 ? acc[t][1] * __expf(c0 - e1) * d1 : 0.f;
                const float m10 = q0 <= i1 ? acc[t][2] * __expf(c1 - e0) * d0 : 0.f, m11 = q1 <= i1 ? acc[t][3] * __expf(c1 - e1) * d1 : 0.f;
                uint32_t hi, lo;
                split_bf16(m00, m01, hi, lo);
                const int o0 = sd_m_offset(mb, t / 2, g, t % 2) + 2 * j, o1 = sd_m_offset(mb, t / 2, g + 8, t % 2) + 2 * j;
                *reinterpret_cast<uint32_t*>(sMh + o0) = hi;
                *reinterpret_cast<uint32_t*>(sMl + o0) = lo;
                split_bf16(m10, m11, hi, lo);
                *reinterpret_cast<uint32_t*>(sMh + o1) = hi;
                *reinterpret_cast<uint32_t*>(sMl + o1) = lo;
            }
        }
        __syncthreads();
        // ---- outputs of this warp's 16 values
        __nv_bfloat16* gy = static_cast<__nv_bfloat16*>(p.y) + ((int64_t)b * p.S + t0) * p.y_ld + h * p.P + v0;
        float y[SD_Q / 16][2][4];                         // [16 tokens][values 0-7 | 8-15 of the warp]
#pragma unroll
        for (int mb = 0; mb < SD_Q / 16; ++mb)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[mb][0][e] = y[mb][1][e] = 0.f;
        const uint32_t ca = uC + ((lane % 16) * LDN + (lane / 16) * 8) * 2;
#pragma unroll
        for (int ks = 0; ks < NP / 16; ++ks) {            // C S: the state's two parts, straight from its accumulators
            uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
            split_bf16(st[2 * ks][0], st[2 * ks][1], h0, l0);
            split_bf16(st[2 * ks + 1][0], st[2 * ks + 1][1], h1, l1);
            split_bf16(st[2 * ks][2], st[2 * ks][3], h2, l2);
            split_bf16(st[2 * ks + 1][2], st[2 * ks + 1][3], h3, l3);
#pragma unroll
            for (int mb = 0; mb < SD_Q / 16; ++mb) {
                uint32_t a0, a1, a2, a3;
                ldmatrix_x4(ca + (mb * 16 * LDN + ks * 16) * 2, a0, a1, a2, a3);
                mma_bf16_16816(y[mb][0], a0, a1, a2, a3, h0, h1);
                mma_bf16_16816(y[mb][1], a0, a1, a2, a3, h2, h3);
                mma_bf16_16816(y[mb][0], a0, a1, a2, a3, l0, l1);
                mma_bf16_16816(y[mb][1], a0, a1, a2, a3, l2, l3);
            }
        }
#pragma unroll
        for (int mb = 0; mb < SD_Q / 16; ++mb) {
            const float e0 = expf(s_cum[mb * 16 + g]), e1 = expf(s_cum[mb * 16 + g + 8]);
#pragma unroll
            for (int q = 0; q < 2; ++q) { y[mb][q][0] *= e0; y[mb][q][1] *= e0; y[mb][q][2] *= e1; y[mb][q][3] *= e1; }
        }
#pragma unroll
        for (int ks = 0; ks < SD_Q / 16; ++ks) {          // M x
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(uX + ((ks * 16 + lane % 16) * LDX + warp * 16 + (lane / 16) * 8) * 2, b0, b1, b2, b3);
#pragma unroll
            for (int mb = ks; mb < SD_Q / 16; ++mb) {
                uint32_t a0, a1, a2, a3, d0, d1, d2, d3;
                const uint32_t o = sd_m_offset(mb, ks, lane % 16, lane / 16) * 2;
                ldmatrix_x4(uMh + o, a0, a1, a2, a3);
                ldmatrix_x4(uMl + o, d0, d1, d2, d3);
                mma_bf16_16816(y[mb][0], a0, a1, a2, a3, b0, b1);
                mma_bf16_16816(y[mb][1], a0, a1, a2, a3, b2, b3);
                mma_bf16_16816(y[mb][0], d0, d1, d2, d3, b0, b1);
                mma_bf16_16816(y[mb][1], d0, d1, d2, d3, b2, b3);
            }
        }
        // + D x, rounded; a lane has tokens g and g + 8 of each 16 and values 2 j, 2 j + 1 of each 8
#pragma unroll
        for (int mb = 0; mb < SD_Q / 16; ++mb)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int i = mb * 16 + g + half * 8;
#pragma unroll
                for (int q = 0; q < 2; ++q) {
                    const int v = warp * 16 + q * 8 + 2 * j;
                    if (i < nt && v < nv) {
                        const uint32_t x2 = *reinterpret_cast<const uint32_t*>(sX + i * LDX + v);
                        *reinterpret_cast<uint32_t*>(gy + (int64_t)i * p.y_ld + v) =
                            pack_bf16(fmaf(D, bf16_lo(x2), y[mb][q][half * 2]), fmaf(D, bf16_hi(x2), y[mb][q][half * 2 + 1]));
                    }
                }
            }
        // ---- state: S^T (values x N) = e^{c_last} S^T + (w x)^T B
        const float decay = expf(s_cum[SD_Q - 1]);
#pragma unroll
        for (int t = 0; t < NP / 8; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) st[t][e] *= decay;
#pragma unroll 1
        for (int ks = 0; ks < SD_Q / 16; ++ks) {
            // A fragment: rows = values, columns = tokens; x is stored (token, value), so the load transposes.
            // Matrices: (tokens 0-7 | 8-15) x (values 0-7 | 8-15) -> a0: values lo, tokens lo; a1: values hi, tokens lo; ...
            uint32_t x0, x1, x2, x3;
            ldmatrix_x4_trans(uX + ((ks * 16 + (lane / 16) * 8 + lane % 8) * LDX + warp * 16 + (lane / 8 % 2) * 8) * 2, x0, x1, x2, x3);
            const float w0 = s_w[ks * 16 + 2 * j], w1 = s_w[ks * 16 + 2 * j + 1];
            const float w2 = s_w[ks * 16 + 8 + 2 * j], w3 = s_w[ks * 16 + 8 + 2 * j + 1];
            uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
            split_bf16(bf16_lo(x0) * w0, bf16_hi(x0) * w1, h0, l0);
            split_bf16(bf16_lo(x1) * w0, bf16_hi(x1) * w1, h1, l1);
            split_bf16(bf16_lo(x2) * w2, bf16_hi(x2) * w3, h2, l2);
            split_bf16(bf16_lo(x3) * w2, bf16_hi(x3) * w3, h3, l3);
#pragma unroll
            for (int t2 = 0; t2 < NP / 16; ++t2) {
                uint32_t b0, b1, b2, b3;                  // rows = tokens, columns = state: transposing load
                ldmatrix_x4_trans(uB + ((ks * 16 + lane % 16) * LDN + t2 * 16 + (lane / 16) * 8) * 2, b0, b1, b2, b3);
                mma_bf16_16816(st[2 * t2], h0, h1, h2, h3, b0, b1);
                mma_bf16_16816(st[2 * t2 + 1], h0, h1, h2, h3, b2, b3);
                mma_bf16_16816(st[2 * t2], l0, l1, l2, l3, b0, b1);
                mma_bf16_16816(st[2 * t2 + 1], l0, l1, l2, l3, b2, b3);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < NP / 8; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = g + (e / 2) * 8, n = t * 8 + 2 * j + e % 2;
            if (warp * 16 + r < nv && n < p.N) state[(int64_t)r * p.N + n] = st[t][e];
        }
}

bool ssd_scan_ok(const SsmScanParams& p) {
    return p.N % 8 == 0 && p.N <= 128 && p.P % 8 == 0 && p.xbc_ld % 8 == 0 && p.y_ld % 2 == 0 && (p.H * p.P) % 8 == 0 &&
           ((reinterpret_cast<uintptr_t>(p.xbc) | reinterpret_cast<uintptr_t>(p.y)) & 15) == 0;
}

template <int NP>
static int ssd_launch(const SsmScanParams& p, int W, cudaStream_t st) {
    const int PW = W * 16, slices = (p.P + PW - 1) / PW;
    const size_t smem = (size_t)(2 * SD_Q * (NP + 8) + 2 * SD_MBLOCKS * 256 + SD_Q * (PW + 8)) * 2 + 3 * SD_Q * 4;
    int dev = 0;
    cudaGetDevice(&dev);
    static thread_local int configured_dev = -1;
    if (configured_dev != dev) {
        cudaError_t e = cudaFuncSetAttribute(ssd_scan_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024);
        if (e != cudaSuccess) return fail(BN_ERR_CUDA, "bn_ssm_scan: %s", cudaGetErrorString(e));
        configured_dev = dev;
    }
    launch_dependent(ssd_scan_kernel<NP>, (unsigned)((long long)p.B * p.H * slices), W * 32, smem, st, p, slices);
    return launch_status("bn_ssm_scan");
}

int ssd_scan(const SsmScanParams& p, cudaStream_t st) {
    // a head's values over as few CTAs as four warps allow, evenly: the 64 x 64 matrix is worked out once per CTA
    const int tiles = (p.P + 15) / 16, slices = (tiles + 3) / 4, W = (tiles + slices - 1) / slices;
    if (p.N <= 16) return ssd_launch<16>(p, W, st);
    if (p.N <= 32) return ssd_launch<32>(p, W, st);
    if (p.N <= 64) return ssd_launch<64>(p, W, st);
    return ssd_launch<128>(p, W, st);
}

}  // namespace bn
