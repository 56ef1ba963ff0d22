// Latent attention with a sliding window: keys and values of a token are expanded from one normalised latent vector c
// (kv_rank wide) plus one rotated key part (rot wide) that all heads share, so those two are all that is cached.
//
//   prompt portions   the latents of the window before the portion are gathered from the cache in front of the
//                     portion's own, both are expanded by ONE product to per-head keys and values, and attention runs
//                     over those rows                               (bn_latent_prep, bn_latent_gather, bn_attn_window)
//   one new token     the key expansion moves to the query side, q_c = W_uk^T q, so scores are taken against the cached
//                     latents themselves; the weighted sum of latents is expanded once at the end
//                                                     (bn_latent_absorb_q, bn_latent_decode, bn_latent_expand_out)
//
// Cache: ring[slot][ring_tokens][c: kv_ld | rotated key part: rot_ld], the token of position p at row p % ring_tokens,
// ring_tokens >= window: what the window has passed is overwritten.  kv_ld and rot_ld are kv_rank and rot rounded up to
// multiples of 8; the columns in between hold zeros, in the ring and in every buffer of the same shape, so products and
// dot products may run over them.
//
// The kernels of this file take any sizes, in fp32 and in bf16; the tensor-core forms for the common sizes are in
// latent_decode.cu, attention over expanded keys is in attn_portion.cu.
#include "common.cuh"
#include "hybrid.cuh"
#include "latent.cuh"

namespace bn {

// ---------------------------------------------------------------------------------------------------------------
// One row of the down projections [c_q: q_rank | c: kv_rank | k_rot: rot] -> normalised c_q, normalised c, rotated
// k_rot, and the last two into the cache
// ---------------------------------------------------------------------------------------------------------------
struct LatentPrepParams {
    const void* proj;
    int64_t proj_ld;
    const float *q_norm, *kv_norm;
    const double* freq;
    const int32_t *seq_ids, *positions;
    void *cq, *c, *krot, *ring;
    int64_t cq_ld;
    int rows, S, q_rank, kv_rank, rot, kv_ld, rot_ld, rows_per_seq, row_offset, ring_tokens;
    float eps;
};

constexpr int LP_THREADS = 128;

// VEC = 4: ranks and row strides are multiples of 4 and every row starts on a 16-byte (bf16: 8-byte) boundary
template <typename T, int VEC>
__global__ void __launch_bounds__(LP_THREADS)
latent_prep_kernel(const LatentPrepParams p) {
    __shared__ float sh[2][LP_THREADS / 32];
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    for (int r = blockIdx.x; r < p.rows; r += gridDim.x) {
        const int b = r / p.S, s = r - b * p.S;
        const T* in = static_cast<const T*>(p.proj) + (int64_t)r * p.proj_ld;
        float sq = 0.f, sk = 0.f;
        auto sum_squares = [&](const T* x, int n) {
            float s = 0.f;
            if (VEC == 4) {
#pragma unroll 4
                for (int i = threadIdx.x * 4; i < n; i += LP_THREADS * 4) {
                    float v[4];
                    load4(x + i, v);
#pragma unroll
                    for (int e = 0; e < 4; ++e) s = fmaf(v[e], v[e], s);
                }
            } else {
                for (int i = threadIdx.x; i < n; i += LP_THREADS) { const float v = to_f(x[i]); s = fmaf(v, v, s); }
            }
            return s;
        };
        sq = sum_squares(in, p.q_rank);
        sk = sum_squares(in + p.q_rank, p.kv_rank);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            sq += __shfl_xor_sync(0xffffffffu, sq, o);
            sk += __shfl_xor_sync(0xffffffffu, sk, o);
        }
        __syncthreads();
        if (threadIdx.x % 32 == 0) { sh[0][threadIdx.x / 32] = sq; sh[1][threadIdx.x / 32] = sk; }
        __syncthreads();
        sq = sk = 0.f;
#pragma unroll
        for (int w = 0; w < LP_THREADS / 32; ++w) { sq += sh[0][w]; sk += sh[1][w]; }
        const float inv_q = rsqrtf(sq / (float)p.q_rank + p.eps), inv_k = rsqrtf(sk / (float)p.kv_rank + p.eps);

        // n of ld columns normalised, the rest zero, to one or two places
        auto emit = [&](const T* x, float inv, const float* w, int n, int ld, T* d0, T* d1) {
            if (VEC == 4) {
#pragma unroll 4
                for (int i = threadIdx.x * 4; i < ld; i += LP_THREADS * 4) {
                    float v[4] = {0.f, 0.f, 0.f, 0.f};
                    if (i < n) {
                        float w4[4];
                        load4(x + i, v);
                        load4(w + i, w4);
#pragma unroll
                        for (int e = 0; e < 4; ++e) v[e] = v[e] * inv * w4[e];
                    }
                    if (d0) store4(d0 + i, v);
                    if (d1) store4(d1 + i, v);
                }
            } else {
                for (int i = threadIdx.x; i < ld; i += LP_THREADS) {
                    const T v = from_f<T>(i < n ? to_f(x[i]) * inv * w[i] : 0.f);
                    if (d0) d0[i] = v;
                    if (d1) d1[i] = v;
                }
            }
        };
        T* cq = static_cast<T*>(p.cq) + (int64_t)r * p.cq_ld;
        emit(in, inv_q, p.q_norm, p.q_rank, (int)p.cq_ld, cq, nullptr);

        const int pos = p.positions[b] + s;
        const int64_t out_row = (int64_t)b * p.rows_per_seq + p.row_offset + s;
        T* c = p.c ? static_cast<T*>(p.c) + out_row * p.kv_ld : nullptr;
        T* kr = p.krot ? static_cast<T*>(p.krot) + out_row * p.rot_ld : nullptr;
        // of a portion longer than the ring only the last ring_tokens rows are kept, so no ring row is written twice
        T* ring = nullptr;
        if (p.ring && s >= p.S - p.ring_tokens) {
            const int slot = p.seq_ids ? p.seq_ids[b] : b;
            ring = static_cast<T*>(p.ring) + ((int64_t)slot * p.ring_tokens + pos % p.ring_tokens) * (p.kv_ld + p.rot_ld);
        }
        emit(in + p.q_rank, inv_k, p.kv_norm, p.kv_rank, p.kv_ld, c, ring);
        const T* rin = in + p.q_rank + p.kv_rank;
        for (int i = threadIdx.x; i < p.rot_ld / 2; i += LP_THREADS) {
            T lo = from_f<T>(0.f), hi = lo;
            if (2 * i < p.rot) {
                const float u = to_f(rin[2 * i]), v = to_f(rin[2 * i + 1]);
                float cs, sn;
                rotation(pos, p.freq[i], &cs, &sn);
                lo = from_f<T>(u * cs - v * sn);
                hi = from_f<T>(v * cs + u * sn);
            }
            if (kr) { kr[2 * i] = lo; kr[2 * i + 1] = hi; }
            if (ring) { ring[p.kv_ld + 2 * i] = lo; ring[p.kv_ld + 2 * i + 1] = hi; }
        }
    }
}

// The same with a row held in registers: cq_ld <= 512 NQ, kv_ld <= 512 NK, ranks and strides multiples of 4, rows aligned,
// rot <= 2 LP_THREADS.
// Everything a row needs is requested before the sums.
template <typename T, int NQ, int NK>
__global__ void __launch_bounds__(LP_THREADS, 8)
latent_prep_regs_kernel(const LatentPrepParams p) {
    __shared__ float sh[2][LP_THREADS / 32];
    const int tid = threadIdx.x;
    const double freq = 2 * tid < p.rot ? p.freq[tid] : 0.0;
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    for (int r = blockIdx.x; r < p.rows; r += gridDim.x) {
        const int b = r / p.S, s = r - b * p.S;
        const T* in = static_cast<const T*>(p.proj) + (int64_t)r * p.proj_ld;
        const T* rin = in + p.q_rank + p.kv_rank;
        float vq[NQ][4], vk[NK][4], u = 0.f, v = 0.f;
#pragma unroll
        for (int k = 0; k < NQ; ++k) {
            vq[k][0] = vq[k][1] = vq[k][2] = vq[k][3] = 0.f;
            if ((tid + k * LP_THREADS) * 4 < p.q_rank) load4(in + (tid + k * LP_THREADS) * 4, vq[k]);
        }
#pragma unroll
        for (int k = 0; k < NK; ++k) {
            vk[k][0] = vk[k][1] = vk[k][2] = vk[k][3] = 0.f;
            if ((tid + k * LP_THREADS) * 4 < p.kv_rank) load4(in + p.q_rank + (tid + k * LP_THREADS) * 4, vk[k]);
        }
        if (2 * tid < p.rot) { u = to_f(rin[2 * tid]); v = to_f(rin[2 * tid + 1]); }
        const int pos = p.positions[b] + s, slot = p.seq_ids ? p.seq_ids[b] : b;
        float cs = 1.f, sn = 0.f;
        if (2 * tid < p.rot) rotation(pos, freq, &cs, &sn);      // while the row is on its way
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int k = 0; k < NQ; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) sq = fmaf(vq[k][e], vq[k][e], sq);
#pragma unroll
        for (int k = 0; k < NK; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) sk = fmaf(vk[k][e], vk[k][e], sk);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            sq += __shfl_xor_sync(0xffffffffu, sq, o);
            sk += __shfl_xor_sync(0xffffffffu, sk, o);
        }
        __syncthreads();
        if (tid % 32 == 0) { sh[0][tid / 32] = sq; sh[1][tid / 32] = sk; }
        __syncthreads();
        sq = sk = 0.f;
#pragma unroll
        for (int w = 0; w < LP_THREADS / 32; ++w) { sq += sh[0][w]; sk += sh[1][w]; }
        const float inv_q = rsqrtf(sq / (float)p.q_rank + p.eps), inv_k = rsqrtf(sk / (float)p.kv_rank + p.eps);
        T* cq = static_cast<T*>(p.cq) + (int64_t)r * p.cq_ld;
        const int64_t out_row = (int64_t)b * p.rows_per_seq + p.row_offset + s;
        T* c = p.c ? static_cast<T*>(p.c) + out_row * p.kv_ld : nullptr;
        T* kr = p.krot ? static_cast<T*>(p.krot) + out_row * p.rot_ld : nullptr;
        T* ring = nullptr;
        if (p.ring && s >= p.S - p.ring_tokens)
            ring = static_cast<T*>(p.ring) + ((int64_t)slot * p.ring_tokens + pos % p.ring_tokens) * (p.kv_ld + p.rot_ld);
        const float zero[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int k = 0; k < NQ; ++k) {
            const int i = (tid + k * LP_THREADS) * 4;
            if (i < p.q_rank) {
                float w4[4];
                load4(p.q_norm + i, w4);
#pragma unroll
                for (int e = 0; e < 4; ++e) vq[k][e] = vq[k][e] * inv_q * w4[e];
                store4(cq + i, vq[k]);
            } else if (i < p.cq_ld) store4(cq + i, zero);
        }
#pragma unroll
        for (int k = 0; k < NK; ++k) {
            const int i = (tid + k * LP_THREADS) * 4;
            if (i < p.kv_rank) {
                float w4[4];
                load4(p.kv_norm + i, w4);
#pragma unroll
                for (int e = 0; e < 4; ++e) vk[k][e] = vk[k][e] * inv_k * w4[e];
                if (c) store4(c + i, vk[k]);
                if (ring) store4(ring + i, vk[k]);
            } else if (i < p.kv_ld) {
                if (c) store4(c + i, zero);
                if (ring) store4(ring + i, zero);
            }
        }
        if (2 * tid < p.rot_ld) {
            T lo = from_f<T>(0.f), hi = lo;
            if (2 * tid < p.rot) {
                lo = from_f<T>(u * cs - v * sn);
                hi = from_f<T>(v * cs + u * sn);
            }
            if (kr) { kr[2 * tid] = lo; kr[2 * tid + 1] = hi; }
            if (ring) { ring[p.kv_ld + 2 * tid] = lo; ring[p.kv_ld + 2 * tid + 1] = hi; }
        }
    }
}

// the `n_old` tokens before the portion, out of the ring, to rows 0 .. n_old - 1 of each sequence's block of rows
template <typename T>
__global__ void __launch_bounds__(128)
latent_gather_kernel(const T* ring, int ring_tokens, int kv_ld, int rot_ld, const int32_t* seq_ids, const int32_t* positions,
                     int B, int n_old, T* c, T* krot, int rows_per_seq) {
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    for (int r = blockIdx.x; r < B * n_old; r += gridDim.x) {
        const int b = r / n_old, i = r - b * n_old;
        const int pos = positions[b] - n_old + i;
        if (pos < 0) continue;                         // the host sized n_old by the same positions
        const int slot = seq_ids ? seq_ids[b] : b;
        const T* src = ring + ((int64_t)slot * ring_tokens + pos % ring_tokens) * (kv_ld + rot_ld);
        T* cd = c + ((int64_t)b * rows_per_seq + i) * kv_ld;
        T* kd = krot + ((int64_t)b * rows_per_seq + i) * rot_ld;
        for (int j = threadIdx.x; j < kv_ld; j += 128) cd[j] = src[j];
        for (int j = threadIdx.x; j < rot_ld; j += 128) kd[j] = src[kv_ld + j];
    }
}

// rotates, in place, the last `rot` of each head's `dim + rot` columns
template <typename T>
__global__ void __launch_bounds__(256)
rope_heads_kernel(T* q, int64_t q_ld, long long n, int S, int H, int dim, int rot, const double* freq, const int32_t* positions) {
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int half = rot / 2;
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) {
        // n = rows * half pairs: a thread turns one pair of one row in every head, with one sine and cosine
        const int64_t r = i / half;
        const int j = (int)(i - r * half);
        float cs, sn;
        rotation(positions[r / S] + (int)(r % S), freq[j], &cs, &sn);
        T* x = q + r * q_ld + dim + 2 * j;
        for (int h = 0; h < H; ++h, x += dim + rot) {
            const float u = to_f(x[0]), v = to_f(x[1]);
            x[0] = from_f<T>(u * cs - v * sn);
            x[1] = from_f<T>(v * cs + u * sn);
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------
// One new token per row: the query moved into latent space.  Block (row group, n tile, head); the last n tile is the
// rotation.
//   q_abs[b][h][0..kv_ld) = sum_i q[b][h][i] W_uk[h * dim + i][:]      q_abs[b][h][kv_ld..) = rotated part
// ---------------------------------------------------------------------------------------------------------------
constexpr int LA_N = 128, LA_B = 8;

template <typename T>
__global__ void __launch_bounds__(LA_N)
latent_absorb_kernel(const T* q, int64_t q_ld, const T* wuk, const double* freq, const int32_t* positions, T* q_abs, int B, int H,
                     int dim, int rot, int kv_ld, int rot_ld) {
    extern __shared__ __align__(16) float qa_smem[];    // [dim][LA_B]
    float* q_smem = qa_smem;
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int n_tiles = (kv_ld + LA_N - 1) / LA_N, h = blockIdx.x % H, tile = blockIdx.x / H % (n_tiles + 1);
    const int b0 = blockIdx.x / (H * (n_tiles + 1)) * LA_B, nb = min(LA_B, B - b0);
    const int width = kv_ld + rot_ld;
    if (tile == n_tiles) {
        for (int i = threadIdx.x; i < nb * (rot_ld / 2); i += LA_N) {
            const int b = b0 + i / (rot_ld / 2), j = i % (rot_ld / 2);
            T lo = from_f<T>(0.f), hi = lo;
            if (2 * j < rot) {
                const T* x = q + b * q_ld + h * (dim + rot) + dim + 2 * j;
                const float u = to_f(x[0]), v = to_f(x[1]);
                float cs, sn;
                rotation(positions[b], freq[j], &cs, &sn);
                lo = from_f<T>(u * cs - v * sn);
                hi = from_f<T>(v * cs + u * sn);
            }
            T* o = q_abs + ((int64_t)b * H + h) * width + kv_ld + 2 * j;
            o[0] = lo;
            o[1] = hi;
        }
        return;
    }
    const int n = tile * LA_N + threadIdx.x;
    for (int i = threadIdx.x; i < LA_B * dim; i += LA_N) {
        const int b = i / dim, e = i - b * dim;
        q_smem[e * LA_B + b] = b < nb ? to_f(q[(b0 + b) * q_ld + h * (dim + rot) + e]) : 0.f;
    }
    __syncthreads();
    if (n >= kv_ld) return;
    float acc[LA_B];
#pragma unroll
    for (int b = 0; b < LA_B; ++b) acc[b] = 0.f;
    const T* w = wuk + (int64_t)h * dim * kv_ld + n;
#pragma unroll 16
    for (int e = 0; e < dim; ++e) {
        const float wv = to_f(w[(int64_t)e * kv_ld]);
        float q8[LA_B];
        load4(q_smem + e * LA_B, *reinterpret_cast<float(*)[4]>(q8));
        load4(q_smem + e * LA_B + 4, *reinterpret_cast<float(*)[4]>(q8 + 4));
#pragma unroll
        for (int b = 0; b < LA_B; ++b) acc[b] = fmaf(q8[b], wv, acc[b]);
    }
#pragma unroll
    for (int b = 0; b < LA_B; ++b)
        if (b < nb) q_abs[((int64_t)(b0 + b) * H + h) * width + n] = from_f<T>(acc[b]);
}

// ---------------------------------------------------------------------------------------------------------------
// Scores and weighted latent sum over the ring, any sizes.  Block (row, head, split); warps take 32 keys at a time.
// The partial result of a split is the normalised sum and its log-sum-exp.
// ---------------------------------------------------------------------------------------------------------------
constexpr int LD_WARPS = 4, LD_MAXN = 32;              // kv_ld <= 1024

template <typename T>
__global__ void __launch_bounds__(LD_WARPS * 32)
latent_decode_any_kernel(const LatentDecodeParams p) {
    extern __shared__ float smem[];
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int width = p.kv_ld + p.rot_ld;
    float* qs = smem;                                   // [width]
    float* s_acc = smem + width;                        // [LD_WARPS][kv_ld]
    float* s_ml = s_acc + LD_WARPS * p.kv_ld;           // [LD_WARPS][2]
    const int split = blockIdx.x % p.splits, h = (blockIdx.x / p.splits) % p.H, b = blockIdx.x / (p.splits * p.H);
    const int pos = p.positions[b], slot = p.seq_ids ? p.seq_ids[b] : b;
    const T* q = static_cast<const T*>(p.q_abs) + ((int64_t)b * p.H + h) * width;
    for (int e = threadIdx.x; e < width; e += blockDim.x) qs[e] = to_f(q[e]);
    __syncthreads();
    const int first = max(0, pos - p.window + 1), count = pos - first + 1;
    const int per = ((count + p.splits - 1) / p.splits + 31) / 32 * 32;
    const int k_begin = first + split * per, k_end = min(pos + 1, k_begin + per);
    const T* ring = static_cast<const T*>(p.ring) + (int64_t)slot * p.ring_tokens * width;
    float m = -INFINITY, l = 0.f, acc[LD_MAXN];
#pragma unroll
    for (int v = 0; v < LD_MAXN; ++v) acc[v] = 0.f;
    for (int k0 = k_begin + warp * 32; k0 < k_end; k0 += LD_WARPS * 32) {
        const int k = k0 + lane;
        float sc = -INFINITY;
        if (k < k_end) {
            const T* row = ring + (int64_t)(k % p.ring_tokens) * width;
            float d = 0.f;
            for (int e = 0; e < width; ++e) d = fmaf(qs[e], to_f(row[e]), d);
            sc = d * p.scale;
        }
        float mx = sc;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_new = fmaxf(m, mx), shrink = expf(m - m_new), w = expf(sc - m_new);
        float sum = w;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        l = l * shrink + sum;
        m = m_new;
#pragma unroll
        for (int v = 0; v < LD_MAXN; ++v) acc[v] *= shrink;
        const int nk = min(32, k_end - k0);
        for (int j = 0; j < nk; ++j) {
            const float wj = __shfl_sync(0xffffffffu, w, j);
            const T* row = ring + (int64_t)((k0 + j) % p.ring_tokens) * width;
#pragma unroll
            for (int v = 0; v < LD_MAXN; ++v)
                if (v * 32 + lane < p.kv_ld) acc[v] = fmaf(wj, to_f(row[v * 32 + lane]), acc[v]);
        }
    }
    for (int v = 0; v < LD_MAXN; ++v)
        if (v * 32 + lane < p.kv_ld) s_acc[warp * p.kv_ld + v * 32 + lane] = acc[v];
    if (lane == 0) { s_ml[warp * 2] = m; s_ml[warp * 2 + 1] = l; }
    __syncthreads();
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < LD_WARPS; ++w) M = fmaxf(M, s_ml[w * 2]);
    float L = 0.f, f[LD_WARPS];
#pragma unroll
    for (int w = 0; w < LD_WARPS; ++w) {
        f[w] = M == -INFINITY ? 0.f : expf(s_ml[w * 2] - M);
        L = fmaf(s_ml[w * 2 + 1], f[w], L);
    }
    const int64_t part = ((int64_t)b * p.H + h) * p.splits + split;
    for (int i = threadIdx.x; i < p.kv_ld; i += blockDim.x) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < LD_WARPS; ++w) o = fmaf(s_acc[w * p.kv_ld + i], f[w], o);
        p.partial[part * p.kv_ld + i] = L > 0.f ? o / L : 0.f;
    }
    if (threadIdx.x == 0) p.lse[part] = L > 0.f ? M + logf(L) : -INFINITY;
}

// ---------------------------------------------------------------------------------------------------------------
// Merges the splits and expands the latent sum to the head's values: out[b][h][v] = sum_n W_uv[h * vdim + v][n] o[n].
// Block (value tile of LO_V rows, head, group of LO_B rows); a warp per value row.
// ---------------------------------------------------------------------------------------------------------------
constexpr int LO_WARPS = 8, LO_V = 32, LO_B = 4;

template <typename T>
__global__ void __launch_bounds__(LO_WARPS * 32)
latent_expand_out_kernel(const float* partial, const float* lse, int splits, const T* wuv, T* out, int64_t out_ld, int B, int H,
                         int vdim, int kv_ld) {
    extern __shared__ float o_smem[];                   // [LO_B][kv_ld]
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int v_tiles = (vdim + LO_V - 1) / LO_V;
    const int vt = blockIdx.x % v_tiles, h = (blockIdx.x / v_tiles) % H, b0 = blockIdx.x / (v_tiles * H) * LO_B;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, nb = min(LO_B, B - b0);
    for (int b = 0; b < LO_B; ++b) {
        if (b >= nb) {
            for (int i = threadIdx.x; i < kv_ld; i += blockDim.x) o_smem[b * kv_ld + i] = 0.f;
            continue;
        }
        const int64_t part = ((int64_t)(b0 + b) * H + h) * splits;
        float M = -INFINITY;
        for (int s = 0; s < splits; ++s) M = fmaxf(M, lse[part + s]);
        float L = 0.f;
        for (int s = 0; s < splits; ++s) L += expf(lse[part + s] - M);
        const float inv = 1.f / L;
        for (int i = threadIdx.x; i < kv_ld; i += blockDim.x) {
            float o = 0.f;
            for (int s = 0; s < splits; ++s) o = fmaf(partial[(part + s) * kv_ld + i], expf(lse[part + s] - M), o);
            o_smem[b * kv_ld + i] = o * inv;
        }
    }
    __syncthreads();
    for (int v = vt * LO_V + warp; v < min(vdim, (vt + 1) * LO_V); v += LO_WARPS) {
        const T* w = wuv + ((int64_t)h * vdim + v) * kv_ld;
        float acc[LO_B];
#pragma unroll
        for (int b = 0; b < LO_B; ++b) acc[b] = 0.f;
#pragma unroll 4
        for (int i = lane; i < kv_ld; i += 32) {
            const float wv = to_f(w[i]);
#pragma unroll
            for (int b = 0; b < LO_B; ++b) acc[b] = fmaf(wv, o_smem[b * kv_ld + i], acc[b]);
        }
#pragma unroll
        for (int b = 0; b < LO_B; ++b) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) acc[b] += __shfl_xor_sync(0xffffffffu, acc[b], o);
            if (lane == 0 && b < nb) out[(b0 + b) * out_ld + h * vdim + v] = from_f<T>(acc[b]);
        }
    }
    if (h == H - 1 && vt == 0)                          // the padding columns behind the last head
        for (int b = 0; b < nb; ++b)
            for (int i = H * vdim + threadIdx.x; i < out_ld; i += blockDim.x) out[(b0 + b) * out_ld + i] = from_f<T>(0.f);
}

}  // namespace bn

using namespace bn;

extern "C" int bn_latent_prep(const void* proj, int64_t proj_ld, const float* q_norm, const float* kv_norm, float eps,
                              const double* freq, const int32_t* seq_ids, const int32_t* positions, int B, int S, int q_rank,
                              int kv_rank, int rot, void* cq, int64_t cq_ld, void* c, void* krot, int rows_per_seq,
                              int row_offset, void* ring, int ring_tokens, int dtype, bn_stream_t stream) {
    const char* what = "bn_latent_prep";
    if (!proj || !q_norm || !kv_norm || !freq || !positions || !cq || (!c) != (!krot)) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || S < 0 || q_rank <= 0 || kv_rank <= 0 || rot < 0 || rot % 2 || (ring && ring_tokens <= 0) || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d S=%d q_rank=%d kv_rank=%d rot=%d", what, B, S, q_rank, kv_rank, rot);
    if (int rc = require_sm100()) return rc;
    if (B == 0 || S == 0) return BN_OK;
    LatentPrepParams p{proj, proj_ld, q_norm, kv_norm, freq, seq_ids, positions, cq, c, krot, ring, cq_ld, B * S, S, q_rank,
                       kv_rank, rot, round8(kv_rank), round8(rot), rows_per_seq, row_offset, ring_tokens, eps};
    const int cap = sm_count() * 16;
    const unsigned grid = (unsigned)(B * S < cap ? B * S : cap);
    const uintptr_t all = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q_norm) | reinterpret_cast<uintptr_t>(kv_norm) |
                          reinterpret_cast<uintptr_t>(cq) | reinterpret_cast<uintptr_t>(c) | reinterpret_cast<uintptr_t>(ring);
    const int kl = p.kv_ld;
    const bool vec = q_rank % 4 == 0 && kv_rank % 4 == 0 && proj_ld % 4 == 0 && cq_ld % 4 == 0 && (all & 15) == 0;
    if (dtype == 0 && vec) launch_dependent(latent_prep_kernel<float, 4>, grid, LP_THREADS, 0, as_stream(stream), p);
    else if (dtype == 0) launch_dependent(latent_prep_kernel<float, 1>, grid, LP_THREADS, 0, as_stream(stream), p);
    else if (vec && cq_ld <= 1024 && kl <= 512 && rot <= 2 * LP_THREADS)
        launch_dependent(latent_prep_regs_kernel<__nv_bfloat16, 2, 1>, grid, LP_THREADS, 0, as_stream(stream), p);
    else if (vec && cq_ld <= 2048 && kl <= 1024 && rot <= 2 * LP_THREADS)
        launch_dependent(latent_prep_regs_kernel<__nv_bfloat16, 4, 2>, grid, LP_THREADS, 0, as_stream(stream), p);
    else if (vec) launch_dependent(latent_prep_kernel<__nv_bfloat16, 4>, grid, LP_THREADS, 0, as_stream(stream), p);
    else launch_dependent(latent_prep_kernel<__nv_bfloat16, 1>, grid, LP_THREADS, 0, as_stream(stream), p);
    return launch_status(what);
}

extern "C" int bn_latent_gather(const void* ring, int ring_tokens, int kv_rank, int rot, const int32_t* seq_ids,
                                const int32_t* positions, int B, int n_old, void* c, void* krot, int rows_per_seq, int dtype,
                                bn_stream_t stream) {
    const char* what = "bn_latent_gather";
    if (!ring || !positions || !c || !krot) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || n_old < 0 || n_old > ring_tokens || n_old > rows_per_seq || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d n_old=%d ring_tokens=%d", what, B, n_old, ring_tokens);
    if (int rc = require_sm100()) return rc;
    if (B == 0 || n_old == 0) return BN_OK;
    const long long n = (long long)B * n_old, cap = (long long)sm_count() * 16;
    const unsigned grid = (unsigned)(n < cap ? n : cap);
    const int kl = round8(kv_rank), rl = round8(rot);
    if (dtype == 0)
        launch_dependent(latent_gather_kernel<float>, grid, 128, 0, as_stream(stream), static_cast<const float*>(ring), ring_tokens,
                         kl, rl, seq_ids, positions, B, n_old, static_cast<float*>(c), static_cast<float*>(krot), rows_per_seq);
    else
        launch_dependent(latent_gather_kernel<__nv_bfloat16>, grid, 128, 0, as_stream(stream), static_cast<const __nv_bfloat16*>(ring),
                         ring_tokens, kl, rl, seq_ids, positions, B, n_old, static_cast<__nv_bfloat16*>(c),
                         static_cast<__nv_bfloat16*>(krot), rows_per_seq);
    return launch_status(what);
}

extern "C" int bn_rope_heads(void* q, int64_t q_ld, int B, int S, int H, int dim, int rot, const double* freq,
                             const int32_t* positions, int dtype, bn_stream_t stream) {
    const char* what = "bn_rope_heads";
    if (!q || !freq || !positions) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || S < 0 || H <= 0 || dim < 0 || rot < 0 || rot % 2 || (dtype & ~1)) return fail(BN_ERR_INVALID_ARG, "%s: bad shape", what);
    if (int rc = require_sm100()) return rc;
    const long long n = (long long)B * S * (rot / 2);
    if (n == 0) return BN_OK;
    const long long blocks = (n + 255) / 256, cap = (long long)sm_count() * 32;
    const unsigned grid = (unsigned)(blocks < cap ? blocks : cap);
    if (dtype == 0)
        launch_dependent(rope_heads_kernel<float>, grid, 256, 0, as_stream(stream), static_cast<float*>(q), q_ld, n, S, H, dim, rot,
                         freq, positions);
    else
        launch_dependent(rope_heads_kernel<__nv_bfloat16>, grid, 256, 0, as_stream(stream), static_cast<__nv_bfloat16*>(q), q_ld, n,
                         S, H, dim, rot, freq, positions);
    return launch_status(what);
}

extern "C" int bn_latent_absorb_q(const void* q, int64_t q_ld, const void* wuk, const double* freq, const int32_t* positions,
                                  void* q_abs, int B, int H, int dim, int rot, int kv_rank, int dtype, bn_stream_t stream) {
    const char* what = "bn_latent_absorb_q";
    if (!q || !wuk || !freq || !positions || !q_abs) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || H <= 0 || dim <= 0 || rot < 0 || rot % 2 || kv_rank <= 0 || (dtype & ~1)) return fail(BN_ERR_INVALID_ARG, "%s: bad shape", what);
    if (int rc = require_sm100()) return rc;
    if (B == 0) return BN_OK;
    const int kl = round8(kv_rank), rl = round8(rot);
    if (dtype == 1 && latent_absorb_mma(q, q_ld, wuk, freq, positions, q_abs, B, H, dim, rot, kl, rl, as_stream(stream)))
        return launch_status(what);
    const unsigned grid = (unsigned)(H * ((kl + LA_N - 1) / LA_N + 1) * ((B + LA_B - 1) / LA_B));
    const size_t smem = (size_t)LA_B * dim * sizeof(float);
    if (dtype == 0) {
        if (int rc = allow_smem(latent_absorb_kernel<float>, smem, what)) return rc;
        launch_dependent(latent_absorb_kernel<float>, grid, LA_N, smem, as_stream(stream), static_cast<const float*>(q), q_ld,
                         static_cast<const float*>(wuk), freq, positions, static_cast<float*>(q_abs), B, H, dim, rot, kl, rl);
    } else {
        if (int rc = allow_smem(latent_absorb_kernel<__nv_bfloat16>, smem, what)) return rc;
        launch_dependent(latent_absorb_kernel<__nv_bfloat16>, grid, LA_N, smem, as_stream(stream), static_cast<const __nv_bfloat16*>(q),
                         q_ld, static_cast<const __nv_bfloat16*>(wuk), freq, positions, static_cast<__nv_bfloat16*>(q_abs), B, H, dim,
                         rot, kl, rl);
    }
    return launch_status(what);
}

extern "C" int bn_latent_decode_splits(int B, int H, int kv_rank, int rot, int window, int dtype) {
    if (B <= 0 || H <= 0 || window <= 0) return 0;
    if (dtype == 1 && latent_decode_mma_ok(H, round8(kv_rank), round8(rot))) return latent_decode_mma_splits(B, H, window, sm_count());
    long long want = (2LL * sm_count() + (long long)B * H - 1) / ((long long)B * H);
    const long long most = (window + 127) / 128;
    if (want > most) want = most;
    return (int)(want < 1 ? 1 : want);
}

extern "C" int bn_latent_decode(const void* q_abs, const void* ring, int num_slots, int ring_tokens, const int32_t* seq_ids,
                                const int32_t* positions, float* partial, float* lse, int splits, int B, int H, int kv_rank, int rot,
                                int window, float scale, int dtype, bn_stream_t stream) {
    const char* what = "bn_latent_decode";
    if (!q_abs || !ring || !positions || !partial || !lse) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || H <= 0 || kv_rank <= 0 || rot < 0 || window <= 0 || num_slots <= 0 || ring_tokens < window || splits <= 0 || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d H=%d kv_rank=%d window=%d ring_tokens=%d", what, B, H, kv_rank, window, ring_tokens);
    if (int rc = require_sm100()) return rc;
    if (B == 0) return BN_OK;
    LatentDecodeParams p{q_abs, ring, seq_ids, positions, partial, lse, B, H, round8(kv_rank), round8(rot), num_slots, ring_tokens, window, splits, scale};
    if (dtype == 1 && latent_decode_mma_ok(H, p.kv_ld, p.rot_ld)) return latent_decode_mma(p, as_stream(stream));
    if (p.kv_ld > LD_MAXN * 32) return fail(BN_ERR_UNSUPPORTED, "%s: kv_rank=%d (at most %d)", what, kv_rank, LD_MAXN * 32);
    const size_t smem = (size_t)(p.kv_ld + p.rot_ld + LD_WARPS * p.kv_ld + LD_WARPS * 2) * sizeof(float);
    const unsigned grid = (unsigned)((long long)B * H * splits);
    if (dtype == 0) {
        if (int rc = allow_smem(latent_decode_any_kernel<float>, smem, what)) return rc;
        launch_dependent(latent_decode_any_kernel<float>, grid, LD_WARPS * 32, smem, as_stream(stream), p);
    } else {
        if (int rc = allow_smem(latent_decode_any_kernel<__nv_bfloat16>, smem, what)) return rc;
        launch_dependent(latent_decode_any_kernel<__nv_bfloat16>, grid, LD_WARPS * 32, smem, as_stream(stream), p);
    }
    return launch_status(what);
}

extern "C" int bn_latent_expand_out(float* partial, const float* lse, int splits, const void* wuv, void* out, int64_t out_ld,
                                    int B, int H, int vdim, int kv_rank, int dtype, bn_stream_t stream) {
    const char* what = "bn_latent_expand_out";
    if (!partial || !lse || !wuv || !out) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || H <= 0 || vdim <= 0 || kv_rank <= 0 || splits <= 0 || (dtype & ~1)) return fail(BN_ERR_INVALID_ARG, "%s: bad shape", what);
    if (int rc = require_sm100()) return rc;
    if (B == 0) return BN_OK;
    const int kl = round8(kv_rank);
    if (dtype == 1 && latent_expand_mma(partial, lse, splits, wuv, out, out_ld, B, H, vdim, kl, as_stream(stream)))
        return launch_status(what);
    const unsigned grid = (unsigned)(((vdim + LO_V - 1) / LO_V) * H * ((B + LO_B - 1) / LO_B));
    const size_t smem = (size_t)LO_B * kl * sizeof(float);
    if (dtype == 0) {
        if (int rc = allow_smem(latent_expand_out_kernel<float>, smem, what)) return rc;
        launch_dependent(latent_expand_out_kernel<float>, grid, LO_WARPS * 32, smem, as_stream(stream), partial, lse, splits,
                         static_cast<const float*>(wuv), static_cast<float*>(out), out_ld, B, H, vdim, kl);
    } else {
        if (int rc = allow_smem(latent_expand_out_kernel<__nv_bfloat16>, smem, what)) return rc;
        launch_dependent(latent_expand_out_kernel<__nv_bfloat16>, grid, LO_WARPS * 32, smem, as_stream(stream), partial, lse, splits,
                         static_cast<const __nv_bfloat16*>(wuv), static_cast<__nv_bfloat16*>(out), out_ld, B, H, vdim, kl);
    }
    return launch_status(what);
}
