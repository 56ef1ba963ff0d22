// Mamba-2 mixer between its two products: causal convolution, selective state-space recurrence, gated group norm.
//
//   in-projection row   [z: inner | x: inner | B: G*N | C: G*N | dt: H]      inner = H * P
//   conv                x, B, C through a causal convolution per channel (`taps` taps, bias), then silu
//   step                dt = softplus(dt + dt_bias), a = -exp(A_log) dt
//   recurrence          S = e^a S + dt B x^T per head (S: N x P, fp32), y = S^T C + D x; head h uses group h / (H/G)
//   gate and norm       y * silu(z), RMS-normed in equal parts, times a weight
//
// Per sequence the state is S, kept as [slot][H][P][N] fp32 (N contiguous), and the convolution's last inputs, kept as a
// ring [slot][taps][channels] in which the input of position p sits in row p % taps.  A zeroed slot is a new sequence.
//
// One new token: ONE launch does convolution, step, recurrence and gate (bn_mamba2_step).  It writes row p % taps of the
// ring, the only row that no other block of the launch reads.  A prompt portion: convolution and step over all rows, the
// ring update, the scan, the gated norm.  The scan of this file goes token by token and takes any sizes in fp32 and bf16;
// the chunked tensor-core scan is in ssd_scan.cu.
#include "common.cuh"
#include "hybrid.cuh"
#include "mamba2.cuh"

namespace bn {

// ---------------------------------------------------------------------------------------------------------------
// Convolution + silu of a portion.  A thread owns VEC neighbouring channels over CV_TOK tokens, with the last taps - 1
// inputs in registers.
// ---------------------------------------------------------------------------------------------------------------
struct ConvParams {
    const void* proj;                 // row stride proj_ld; the convolved channels start at column first_col
    const float *w, *bias;            // [C][taps], [C]
    const float *dt_bias, *a_log;     // [H]
    const void* ring;
    const int32_t *seq_ids, *positions;
    void* xbc;                        // (rows, xbc_ld)
    float *dt, *a;                    // (rows, H): step size, log decay
    int64_t proj_ld, xbc_ld;
    int B, S, C, H, taps, first_col;
};

constexpr int CV_TOK = 32, CV_MAXTAPS = 16;

template <typename T, int VEC> struct ConvVec;
template <> struct ConvVec<float, 1> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[1]) { v[0] = *p; }
    static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
};
template <> struct ConvVec<__nv_bfloat16, 1> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[1]) { v[0] = to_f(*p); }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[1]) { *p = from_f<__nv_bfloat16>(v[0]); }
};
template <> struct ConvVec<__nv_bfloat16, 2> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[2]) {
        const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
        v[0] = ptx::bf16_lo(u);
        v[1] = ptx::bf16_hi(u);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[2]) {
        *reinterpret_cast<uint32_t*>(p) = ptx::pack_bf16(v[0], v[1]);
    }
};

template <> struct ConvVec<__nv_bfloat16, 4> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) { load4(p, v); }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) { store4(p, v); }
};

// silu for the bf16 path: its result is rounded to bf16, so the fast exponential is far more exact than needed
template <typename T> __device__ __forceinline__ float conv_silu_f(float z) { return silu_exact(z); }
template <> __device__ __forceinline__ float conv_silu_f<__nv_bfloat16>(float z) { return activation_fast(BN_ACT_SILU, z); }

// TAPS > 0: known at compile time; 0: p.taps (at most CV_MAXTAPS)
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128)
conv_silu_kernel(const ConvParams p) {
    using V = ConvVec<T, VEC>;
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int taps = TAPS ? TAPS : p.taps;
    constexpr int W = TAPS ? TAPS : CV_MAXTAPS;
    const int segs = (p.S + CV_TOK - 1) / CV_TOK;
    const int b = blockIdx.y / segs, t0 = (blockIdx.y % segs) * CV_TOK, t1 = min(p.S, t0 + CV_TOK);
    const int c = (blockIdx.x * 128 + threadIdx.x) * VEC;
    const T* in = static_cast<const T*>(p.proj) + (int64_t)b * p.S * p.proj_ld + p.first_col;
    if (c >= p.C) return;
    float w[W][VEC], bias[VEC], hist[W][VEC];          // hist[k]: the input k + 1 tokens back
#pragma unroll
    for (int e = 0; e < VEC; ++e) bias[e] = p.bias[c + e];
#pragma unroll
    for (int k = 0; k < W; ++k)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            w[k][e] = k < taps ? p.w[(int64_t)(c + e) * taps + taps - 1 - k] : 0.f;   // w[k]: the tap k tokens back
            hist[k][e] = 0.f;
        }
    const int pos0 = p.positions[b];
    const T* ring = static_cast<const T*>(p.ring) + (int64_t)(p.seq_ids ? p.seq_ids[b] : b) * taps * p.C + c;
#pragma unroll
    for (int k = 0; k < W; ++k)
        if (k < taps - 1) {
            const int t = t0 - 1 - k;
            if (t >= 0) V::load(in + (int64_t)t * p.proj_ld + c, hist[k]);
            else if (pos0 + t >= 0) V::load(ring + (int64_t)((pos0 + t) % taps) * p.C, hist[k]);
        }
    T* out = static_cast<T*>(p.xbc) + (int64_t)b * p.S * p.xbc_ld + c;
    auto token = [&](int t, const float (&v)[VEC]) {
        float y[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float s = fmaf(v[e], w[0][e], bias[e]);
#pragma unroll
            for (int k = 1; k < W; ++k)
                if (k < taps) s = fmaf(hist[k - 1][e], w[k][e], s);
            y[e] = conv_silu_f<T>(s);
        }
        V::store(out + (int64_t)t * p.xbc_ld, y);
#pragma unroll
        for (int k = W - 1; k > 0; --k)
#pragma unroll
            for (int e = 0; e < VEC; ++e) hist[k][e] = hist[k - 1][e];
#pragma unroll
        for (int e = 0; e < VEC; ++e) hist[0][e] = v[e];
    };
    constexpr int AHEAD = 8;                           // tokens whose loads are in flight together
    int t = t0;
    for (; t + AHEAD <= t1; t += AHEAD) {
        float v[AHEAD][VEC];
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) V::load(in + (int64_t)(t + a) * p.proj_ld + c, v[a]);
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) token(t + a, v[a]);
    }
    for (; t < t1; ++t) {
        float v[VEC];
        V::load(in + (int64_t)t * p.proj_ld + c, v);
        token(t, v);
    }
}

// What else a portion leaves: its last inputs in the ring (after the convolution has read it), and the step size and log
// decay of every token and head.
template <typename T>
__global__ void __launch_bounds__(256)
conv_tail_kernel(const ConvParams p, T* ring) {
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int keep = min(p.S, p.taps);
    const long long n_ring = (long long)p.B * keep * p.C, n = n_ring + (long long)p.B * p.S * p.H;
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) {
        if (i < n_ring) {
            const int c = (int)(i % p.C), k = (int)(i / p.C % keep), b = (int)(i / p.C / keep), t = p.S - keep + k;
            const int slot = p.seq_ids ? p.seq_ids[b] : b;
            ring[((int64_t)slot * p.taps + (p.positions[b] + t) % p.taps) * p.C + c] =
                static_cast<const T*>(p.proj)[((int64_t)b * p.S + t) * p.proj_ld + p.first_col + c];
        } else {
            const long long q = i - n_ring;
            const int64_t row = q / p.H;
            const int h = (int)(q - row * p.H);
            const float d = softplus_exact(to_f(static_cast<const T*>(p.proj)[row * p.proj_ld + p.first_col + p.C + h]) + p.dt_bias[h]);
            p.dt[q] = d;
            p.a[q] = -expf(p.a_log[h]) * d;
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------
// The recurrence of a portion, token by token: block (sequence, head, SC_P values of P); a warp per value, its N state
// elements over the lanes.
// ---------------------------------------------------------------------------------------------------------------
constexpr int SC_WARPS = 8, SC_MAXN = 16;              // N <= 512

template <typename T>
__global__ void __launch_bounds__(SC_WARPS * 32)
ssm_scan_any_kernel(const SsmScanParams p) {
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int p_tiles = (p.P + SC_WARPS - 1) / SC_WARPS;
    const int pt = blockIdx.x % p_tiles, h = (blockIdx.x / p_tiles) % p.H, b = blockIdx.x / (p_tiles * p.H);
    const int v = pt * SC_WARPS + warp;
    if (v >= p.P) return;
    const int g = h / (p.H / p.G), slot = p.seq_ids ? p.seq_ids[b] : b;
    float* state = p.state + (((int64_t)slot * p.H + h) * p.P + v) * p.N;
    float s[SC_MAXN];
#pragma unroll
    for (int i = 0; i < SC_MAXN; ++i) s[i] = i * 32 + lane < p.N ? state[i * 32 + lane] : 0.f;
    const float D = p.D[h];
    for (int t = 0; t < p.S; ++t) {
        const int64_t row = (int64_t)b * p.S + t;
        const T* xbc = static_cast<const T*>(p.xbc) + row * p.xbc_ld;
        const float x = to_f(xbc[h * p.P + v]), dt = p.dt[row * p.H + h], decay = expf(p.a[row * p.H + h]);
        const T* Bt = xbc + p.H * p.P + g * p.N;
        const T* Ct = Bt + p.G * p.N;
        float y = 0.f;
#pragma unroll
        for (int i = 0; i < SC_MAXN; ++i) {
            const int n = i * 32 + lane;
            if (n < p.N) {
                s[i] = fmaf(decay, s[i], dt * to_f(Bt[n]) * x);
                y = fmaf(s[i], to_f(Ct[n]), y);
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        if (lane == 0) static_cast<T*>(p.y)[row * p.y_ld + h * p.P + v] = from_f<T>(fmaf(D, x, y));
    }
#pragma unroll
    for (int i = 0; i < SC_MAXN; ++i)
        if (i * 32 + lane < p.N) state[i * 32 + lane] = s[i];
}

// ---------------------------------------------------------------------------------------------------------------
// One new token per row: block (row, head, tile of values)
// ---------------------------------------------------------------------------------------------------------------
struct StepParams {
    const void* proj;
    const float *conv_w, *conv_b, *dt_bias, *a_log, *D;
    void* ring;
    float* state;
    const int32_t *seq_ids, *positions;
    float* gated;                     // (rows, H*P): (y + D x) silu(z)
    int64_t proj_ld;
    int B, H, P, G, N, taps, p_per_block;
};

constexpr int ST_WARPS = 8;

// What the convolution of one channel needs, loaded before any of it is used
template <typename T, int TAPS>
struct ConvLoads {
    static constexpr int W = TAPS ? TAPS : CV_MAXTAPS;
    T cur, back[W];
    float w[W], bias;

    __device__ __forceinline__ void load(const StepParams& p, const T* in, const T* ring, int c, int C, int pos) {
        const int taps = TAPS ? TAPS : p.taps;
        cur = in[c];
        bias = __ldg(p.conv_b + c);
        if (TAPS == 4) {
            const float4 f = __ldg(reinterpret_cast<const float4*>(p.conv_w) + c);
            w[0] = f.w; w[1] = f.z; w[2] = f.y; w[3] = f.x;
        } else {
#pragma unroll
            for (int k = 0; k < W; ++k) w[k] = k < taps ? __ldg(p.conv_w + (int64_t)c * taps + taps - 1 - k) : 0.f;
        }
#pragma unroll
        for (int k = 1; k < W; ++k)
            back[k] = k < taps && pos >= k ? ring[(int64_t)((pos - k) % taps) * C + c] : from_f<T>(0.f);
    }
    __device__ __forceinline__ float result() const {
        float s = fmaf(to_f(cur), w[0], bias);
#pragma unroll
        for (int k = 1; k < W; ++k) s = fmaf(to_f(back[k]), w[k], s);
        return round_to<T>(conv_silu_f<T>(s));
    }
};

// R = state elements per lane and value (N <= 32 R), VEC = 4: in pieces of 16 bytes (N a multiple of 128)
template <typename T, int R, int VEC, int TAPS>
__global__ void __launch_bounds__(ST_WARPS * 32)
mamba2_step_kernel(const StepParams p) {
    extern __shared__ float sm[];                      // B [N], C [N], x [p_per_block], silu(z) [p_per_block]
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int p_tiles = (p.P + p.p_per_block - 1) / p.p_per_block;
    const int pt = blockIdx.x % p_tiles, h = (blockIdx.x / p_tiles) % p.H, b = blockIdx.x / (p_tiles * p.H);
    const int g = h / (p.H / p.G), slot = p.seq_ids ? p.seq_ids[b] : b, pos = p.positions[b];
    const int inner = p.H * p.P, GN = p.G * p.N, C = inner + 2 * GN;
    const T* row = static_cast<const T*>(p.proj) + (int64_t)b * p.proj_ld;
    const T* in = row + inner;
    T* ring = static_cast<T*>(p.ring) + (int64_t)slot * p.taps * C;
    const int v0 = pt * p.p_per_block, nv = min(p.p_per_block, p.P - v0);
    float* state = p.state + (((int64_t)slot * p.H + h) * p.P + v0) * p.N;
    // the state of this warp's first values is requested before the convolution
    constexpr int U = 4;                               // values in flight per warp
    float s[U][R];
    auto load_state = [&](int v, float (&d)[R]) {
        const float* sv = state + (int64_t)v * p.N;
#pragma unroll
        for (int i = 0; i < R / VEC; ++i) {
            if (VEC == 4) {
                const float4 f = *reinterpret_cast<const float4*>(sv + (i * 32 + lane) * 4);
                d[i * VEC] = f.x; d[i * VEC + 1] = f.y; d[i * VEC + 2] = f.z; d[i * VEC + 3] = f.w;
            } else {
                d[i] = i * 32 + lane < p.N ? sv[i * 32 + lane] : 0.f;
            }
        }
    };
#pragma unroll
    for (int u = 0; u < U; ++u)
        if (warp + u * ST_WARPS < nv) load_state(warp + u * ST_WARPS, s[u]);
    float *sB = sm, *sC = sm + p.N, *sx = sm + 2 * p.N, *sz = sx + p.p_per_block;
    const float raw_dt = to_f(in[C + h]), dt_bias = p.dt_bias[h], a_log = p.a_log[h], D = p.D[h];
    // Every block of a group computes the group's B and C; one of them writes their ring row.  Two channels per thread at
    // a time, all loads of both before the arithmetic of either.
    const bool owner = pt == 0 && h % (p.H / p.G) == 0;
    const int n_conv = 2 * p.N + nv, taps = TAPS ? TAPS : p.taps;
    auto channel = [&](int i) {
        return i < p.N ? inner + g * p.N + i : i < 2 * p.N ? inner + GN + g * p.N + (i - p.N) : h * p.P + v0 + (i - 2 * p.N);
    };
    constexpr int IT = TAPS ? 2 : 1;
    for (int i0 = threadIdx.x; i0 < n_conv; i0 += IT * ST_WARPS * 32) {
        ConvLoads<T, TAPS> ld[IT];
#pragma unroll
        for (int it = 0; it < IT; ++it) {
            const int i = i0 + it * ST_WARPS * 32;
            if (i < n_conv) ld[it].load(p, in, ring, channel(i), C, pos);
        }
#pragma unroll
        for (int it = 0; it < IT; ++it) {
            const int i = i0 + it * ST_WARPS * 32;
            if (i < n_conv) {
                sm[i] = ld[it].result();               // B, C and x lie one behind the other
                if (owner || i >= 2 * p.N) ring[(int64_t)(pos % taps) * C + channel(i)] = ld[it].cur;
            }
        }
    }
    for (int i = threadIdx.x; i < nv; i += ST_WARPS * 32) sz[i] = conv_silu_f<T>(to_f(row[h * p.P + v0 + i]));
    const float dt = softplus_exact(raw_dt + dt_bias), decay = expf(-expf(a_log) * dt);
    __syncthreads();
    float Bv[R], Cv[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int n = VEC == 4 ? ((i / VEC) * 32 + lane) * 4 + i % VEC : i * 32 + lane;
        Bv[i] = n < p.N ? dt * sB[n] : 0.f;
        Cv[i] = n < p.N ? sC[n] : 0.f;
    }
    for (int v = warp; v < nv; v += ST_WARPS * U) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int vu = v + u * ST_WARPS;
            if (vu >= nv) break;
            const float x = sx[vu];
            float y = 0.f;
#pragma unroll
            for (int i = 0; i < R; ++i) {
                s[u][i] = fmaf(decay, s[u][i], Bv[i] * x);
                y = fmaf(s[u][i], Cv[i], y);
            }
            float* sv = state + (int64_t)vu * p.N;
#pragma unroll
            for (int i = 0; i < R / VEC; ++i) {
                if (VEC == 4)
                    *reinterpret_cast<float4*>(sv + (i * 32 + lane) * 4) =
                        make_float4(s[u][i * VEC], s[u][i * VEC + 1], s[u][i * VEC + 2], s[u][i * VEC + 3]);
                else if (i * 32 + lane < p.N) sv[i * 32 + lane] = s[u][i];
            }
            const int next = vu + ST_WARPS * U;
            if (next < nv) load_state(next, s[u]);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
            if (lane == 0) p.gated[(int64_t)b * inner + h * p.P + v0 + vu] = fmaf(D, x, y) * sz[vu];
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------
// y * silu(z) (z null: y is gated already), RMS norm in `groups` equal parts, weight.  Block per (row, part).
// ---------------------------------------------------------------------------------------------------------------
struct GatedNormParams {
    const void *y, *z;
    const float* w;
    void* out;
    int64_t y_ld, z_ld, out_ld;
    int rows, width, groups;
    float eps;
};

constexpr int GN_THREADS = 256;

// RV > 0: the part is held in RV float4 registers a thread (part % 4 == 0, part <= 1024 RV, aligned rows); 0: any shape
template <typename T, typename TY, int RV>
__global__ void __launch_bounds__(GN_THREADS)
gated_norm_kernel(const GatedNormParams p) {
    extern __shared__ float part_buf[];
    __shared__ float sh[GN_THREADS / 32];
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int n = p.width / p.groups;
    for (long long item = blockIdx.x; item < (long long)p.rows * p.groups; item += gridDim.x) {
        const int64_t r = item / p.groups;
        const int c0 = (int)(item % p.groups) * n;
        const TY* y = static_cast<const TY*>(p.y) + r * p.y_ld + c0;
        const T* z = p.z ? static_cast<const T*>(p.z) + r * p.z_ld + c0 : nullptr;
        float s = 0.f;
        float v[RV ? RV : 1][4];
        if (RV) {
#pragma unroll
            for (int k = 0; k < RV; ++k) {
                const int i = (threadIdx.x + k * GN_THREADS) * 4;
                if (i < n) {
                    load4(y + i, v[k]);
                    if (z) {
                        float z4[4];
                        load4(z + i, z4);
#pragma unroll
                        for (int e = 0; e < 4; ++e) v[k][e] *= conv_silu_f<T>(z4[e]);
                    }
#pragma unroll
                    for (int e = 0; e < 4; ++e) s = fmaf(v[k][e], v[k][e], s);
                }
            }
        } else {
            for (int i = threadIdx.x; i < n; i += GN_THREADS) {
                const float q = to_f(y[i]) * (z ? conv_silu_f<T>(to_f(z[i])) : 1.f);
                part_buf[i] = q;
                s = fmaf(q, q, s);
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        __syncthreads();
        if (threadIdx.x % 32 == 0) sh[threadIdx.x / 32] = s;
        __syncthreads();
        s = 0.f;
#pragma unroll
        for (int w = 0; w < GN_THREADS / 32; ++w) s += sh[w];
        const float inv = rsqrtf(s / (float)n + p.eps);
        T* o = static_cast<T*>(p.out) + r * p.out_ld + c0;
        if (RV) {
#pragma unroll
            for (int k = 0; k < RV; ++k) {
                const int i = (threadIdx.x + k * GN_THREADS) * 4;
                if (i < n) {
                    float w4[4], o4[4];
                    load4(p.w + c0 + i, w4);
#pragma unroll
                    for (int e = 0; e < 4; ++e) o4[e] = v[k][e] * inv * w4[e];
                    store4(o + i, o4);
                }
            }
        } else {
            for (int i = threadIdx.x; i < n; i += GN_THREADS) o[i] = from_f<T>(part_buf[i] * inv * p.w[c0 + i]);
        }
        if (item % p.groups == p.groups - 1)           // the padding columns behind the row
            for (int i = p.width + threadIdx.x; i < p.out_ld; i += GN_THREADS) static_cast<T*>(p.out)[r * p.out_ld + i] = from_f<T>(0.f);
    }
}

template <typename T, typename TY>
static int gated_norm_launch(const GatedNormParams& p, bn_stream_t stream) {
    const char* what = "bn_gated_group_norm";
    int dev = 0, sms = 148;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const long long items = (long long)p.rows * p.groups, cap = (long long)sms * 8;
    const unsigned grid = (unsigned)(items < cap ? items : cap);
    const int n = p.width / p.groups;
    const uintptr_t all = reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.z) | reinterpret_cast<uintptr_t>(p.w) |
                          reinterpret_cast<uintptr_t>(p.out);
    const bool vec = n % 4 == 0 && n <= 8192 && p.y_ld % 4 == 0 && p.z_ld % 4 == 0 && p.out_ld % 4 == 0 && (all & 15) == 0;
    cudaStream_t st = as_stream(stream);
    if (vec && n <= 1024) launch_dependent(gated_norm_kernel<T, TY, 1>, grid, GN_THREADS, 0, st, p);
    else if (vec && n <= 4096) launch_dependent(gated_norm_kernel<T, TY, 4>, grid, GN_THREADS, 0, st, p);
    else if (vec) launch_dependent(gated_norm_kernel<T, TY, 8>, grid, GN_THREADS, 0, st, p);
    else {
        const size_t smem = (size_t)n * sizeof(float);
        if (smem > 200 * 1024) return fail(BN_ERR_UNSUPPORTED, "%s: part of %d columns (at most 51200)", what, n);
        if (smem > 48 * 1024) {
            cudaError_t e = cudaFuncSetAttribute(gated_norm_kernel<T, TY, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return fail(BN_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
        }
        launch_dependent(gated_norm_kernel<T, TY, 0>, grid, GN_THREADS, smem, st, p);
    }
    return launch_status(what);
}

template <typename T, int VEC>
static int conv_launch(const ConvParams& p, cudaStream_t st) {
    const int segs = (p.S + CV_TOK - 1) / CV_TOK;
    const dim3 grid((p.C + 128 * VEC - 1) / (128 * VEC), (unsigned)(p.B * segs));
    if (p.taps == 4) conv_silu_kernel<T, VEC, 4><<<grid, 128, 0, st>>>(p);
    else conv_silu_kernel<T, VEC, 0><<<grid, 128, 0, st>>>(p);
    return launch_status("bn_mamba2_conv");
}

template <typename T, int R, int VEC>
static int step_launch_taps(const StepParams& p, cudaStream_t st) {
    const unsigned grid = (unsigned)((long long)p.B * p.H * ((p.P + p.p_per_block - 1) / p.p_per_block));
    const size_t smem = (size_t)(2 * p.N + 2 * p.p_per_block) * sizeof(float);
    if (smem > 48 * 1024) return fail(BN_ERR_UNSUPPORTED, "bn_mamba2_step: vdim=%d", p.P);
    if (p.taps == 4 && (reinterpret_cast<uintptr_t>(p.conv_w) & 15) == 0)
        launch_dependent(mamba2_step_kernel<T, R, VEC, 4>, grid, ST_WARPS * 32, smem, st, p);
    else launch_dependent(mamba2_step_kernel<T, R, VEC, 0>, grid, ST_WARPS * 32, smem, st, p);
    return launch_status("bn_mamba2_step");
}

template <typename T>
static int step_launch(const StepParams& p, cudaStream_t st) {
    if (p.N == 128) return step_launch_taps<T, 4, 4>(p, st);
    if (p.N == 256) return step_launch_taps<T, 8, 4>(p, st);
    if (p.N <= 64) return step_launch_taps<T, 2, 1>(p, st);
    if (p.N <= 256) return step_launch_taps<T, 8, 1>(p, st);
    return step_launch_taps<T, 16, 1>(p, st);
}

}  // namespace bn

using namespace bn;

static int mamba2_shape(const char* what, int B, int S, int H, int P, int G, int N, int taps, int dtype) {
    if (B < 0 || S < 0 || H <= 0 || P <= 0 || G <= 0 || N <= 0 || taps <= 0 || H % G || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d S=%d heads=%d vdim=%d groups=%d state=%d taps=%d", what, B, S, H, P, G, N, taps);
    if (taps > CV_MAXTAPS) return fail(BN_ERR_UNSUPPORTED, "%s: %d taps (at most %d)", what, taps, CV_MAXTAPS);
    if (N > SC_MAXN * 32) return fail(BN_ERR_UNSUPPORTED, "%s: state=%d (at most %d)", what, N, SC_MAXN * 32);
    return require_sm100();
}

extern "C" int bn_mamba2_conv(const void* proj, int64_t proj_ld, const float* conv_w, const float* conv_b, const float* dt_bias,
                              const float* a_log, void* ring, const int32_t* seq_ids, const int32_t* positions, int B, int S,
                              int H, int P, int G, int N, int taps, void* xbc, int64_t xbc_ld, float* dt, float* a, int dtype,
                              bn_stream_t stream) {
    const char* what = "bn_mamba2_conv";
    if (!proj || !conv_w || !conv_b || !dt_bias || !a_log || !ring || !positions || !xbc || !dt || !a)
        return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (int rc = mamba2_shape(what, B, S, H, P, G, N, taps, dtype)) return rc;
    if (B == 0 || S == 0) return BN_OK;
    const int inner = H * P, C = inner + 2 * G * N;
    ConvParams p{proj, conv_w, conv_b, dt_bias, a_log, ring, seq_ids, positions, xbc, dt, a, proj_ld, xbc_ld, B, S, C, H, taps, inner};
    if ((long long)B * ((S + CV_TOK - 1) / CV_TOK) > 65535) return fail(BN_ERR_UNSUPPORTED, "%s: B=%d x S=%d too large", what, B, S);
    cudaStream_t st = as_stream(stream);
    const bool fours = C % 4 == 0 && inner % 4 == 0 && proj_ld % 4 == 0 && xbc_ld % 4 == 0 && taps == 4 &&
                       ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(ring) | reinterpret_cast<uintptr_t>(xbc)) & 7) == 0;
    const bool pairs = C % 2 == 0 && inner % 2 == 0 && proj_ld % 2 == 0 && xbc_ld % 2 == 0 &&
                       ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(ring) | reinterpret_cast<uintptr_t>(xbc)) & 3) == 0;
    int rc;
    if (dtype == 0) rc = conv_launch<float, 1>(p, st);
    else if (fours) rc = conv_launch<__nv_bfloat16, 4>(p, st);
    else if (pairs) rc = conv_launch<__nv_bfloat16, 2>(p, st);
    else rc = conv_launch<__nv_bfloat16, 1>(p, st);
    if (rc) return rc;
    const long long n = (long long)B * (S < taps ? S : taps) * C + (long long)B * S * H, blocks = (n + 255) / 256;
    const unsigned grid = (unsigned)(blocks < 8192 ? blocks : 8192);
    if (dtype == 0) launch_dependent(conv_tail_kernel<float>, grid, 256, 0, st, p, static_cast<float*>(ring));
    else launch_dependent(conv_tail_kernel<__nv_bfloat16>, grid, 256, 0, st, p, static_cast<__nv_bfloat16*>(ring));
    return launch_status(what);
}

extern "C" int bn_ssm_scan(const void* xbc, int64_t xbc_ld, const float* dt, const float* a, const float* D, float* state,
                           const int32_t* seq_ids, int B, int S, int H, int P, int G, int N, void* y, int64_t y_ld, int dtype,
                           bn_stream_t stream) {
    const char* what = "bn_ssm_scan";
    if (!xbc || !dt || !a || !D || !state || !y) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (int rc = mamba2_shape(what, B, S, H, P, G, N, 1, dtype)) return rc;
    if (B == 0 || S == 0) return BN_OK;
    SsmScanParams p{xbc, dt, a, D, state, seq_ids, y, xbc_ld, y_ld, B, S, H, P, G, N};
    if (dtype == 1 && ssd_scan_ok(p)) return ssd_scan(p, as_stream(stream));
    const unsigned grid = (unsigned)((long long)B * H * ((P + SC_WARPS - 1) / SC_WARPS));
    if (dtype == 0) launch_dependent(ssm_scan_any_kernel<float>, grid, SC_WARPS * 32, 0, as_stream(stream), p);
    else launch_dependent(ssm_scan_any_kernel<__nv_bfloat16>, grid, SC_WARPS * 32, 0, as_stream(stream), p);
    return launch_status(what);
}

extern "C" int bn_mamba2_step(const void* proj, int64_t proj_ld, const float* conv_w, const float* conv_b, const float* dt_bias,
                              const float* a_log, const float* D, void* ring, float* state, const int32_t* seq_ids,
                              const int32_t* positions, int B, int H, int P, int G, int N, int taps, float* gated, int dtype,
                              bn_stream_t stream) {
    const char* what = "bn_mamba2_step";
    if (!proj || !conv_w || !conv_b || !dt_bias || !a_log || !D || !ring || !state || !positions || !gated)
        return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (int rc = mamba2_shape(what, B, 1, H, P, G, N, taps, dtype)) return rc;
    if (B == 0) return BN_OK;
    // few rows: a head's values are cut over several blocks, so that the state is moved by the whole GPU
    int dev = 0, sms = 148;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    int per = P;
    while (per > 16 && (long long)B * H * ((P + per - 1) / per) < 4LL * sms) per = (per + 1) / 2;
    StepParams p{proj, conv_w, conv_b, dt_bias, a_log, D, ring, state, seq_ids, positions, gated, proj_ld, B, H, P, G, N, taps, per};
    return dtype == 0 ? step_launch<float>(p, as_stream(stream)) : step_launch<__nv_bfloat16>(p, as_stream(stream));
}

extern "C" int bn_gated_group_norm(const void* y, int64_t y_ld, int y_dtype, const void* z, int64_t z_ld, const float* w, void* out,
                                   int64_t out_ld, int rows, int width, int groups, float eps, int dtype, bn_stream_t stream) {
    const char* what = "bn_gated_group_norm";
    if (!y || !w || !out) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (rows < 0 || width <= 0 || groups <= 0 || width % groups || ((dtype | y_dtype) & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape rows=%d width=%d groups=%d", what, rows, width, groups);
    if (int rc = require_sm100()) return rc;
    if (rows == 0) return BN_OK;
    GatedNormParams p{y, z, w, out, y_ld, z_ld, out_ld, rows, width, groups, eps};
    if (dtype == 0 && y_dtype == 0) return gated_norm_launch<float, float>(p, stream);
    if (dtype == 0) return fail(BN_ERR_UNSUPPORTED, "%s: bf16 input on the fp32 path", what);
    if (y_dtype == 0) return gated_norm_launch<__nv_bfloat16, float>(p, stream);
    return gated_norm_launch<__nv_bfloat16, __nv_bfloat16>(p, stream);
}
