// Attention of a prompt portion (bn_attn_window: a sliding window and a rotated key part shared by the heads;
// bn_attn_chunked: grouped-query heads, chunks of positions, unit-RMS queries, a gate on the result) for any sizes, in fp32
// and in bf16, and the choice of the tensor-core form (attn_portion_sm100.cu).
#include "attn_portion.cuh"
#include "common.cuh"
#include "hybrid.cuh"

namespace bn {

// ---------------------------------------------------------------------------------------------------------------
// Portion attention, and one-token attention over cached keys, any sizes: a warp per (query row, head); 32 keys at a time, a
// lane per key for the scores, then a lane per value column.  Scores, weights and sums in fp32.
// ---------------------------------------------------------------------------------------------------------------
constexpr int AW_WARPS = 4, AW_MAXV = 16;      // vdim <= 512

template <typename T>
__global__ void __launch_bounds__(AW_WARPS * 32)
attn_any_kernel(const AttnPortionParams p) {
    extern __shared__ float q_smem[];
    ptx::grid_dependency_wait();
    ptx::grid_launch_dependents();
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int E = p.dim + p.rot;
    float* qs = q_smem + warp * E;
    const long long n = (long long)p.B * p.S * p.H;
    for (long long item = (long long)blockIdx.x * AW_WARPS + warp; item < n; item += (long long)gridDim.x * AW_WARPS) {
        const int h = (int)(item % p.H);
        const long long row = item / p.H;
        const int b = (int)(row / p.S), s = (int)(row - (long long)b * p.S);
        const T* q = static_cast<const T*>(p.q) + row * p.q_ld + h * E;
        __syncwarp();
        float ss = 0.f;
        for (int e = lane; e < E; e += 32) { qs[e] = to_f(q[e]); ss = fmaf(qs[e], qs[e], ss); }
        __syncwarp();
        float scale = p.scale;
        if (p.rms_dim) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            scale *= rsqrtf(ss / (float)p.rms_dim + p.rms_eps);
        }
        const int g = h / (p.H / p.kv_heads), block = p.seq_ids ? p.seq_ids[b] : b;
        const int last = p.positions ? p.positions[b] % p.span : p.n_old + s, first = max(0, mask_oldest(p.mask, p.span, last));
        if (p.positions && last >= p.rows_per_seq) {       // the cache has no room for this token
            for (int v = lane; v < p.vdim; v += 32)
                static_cast<T*>(p.out)[row * p.out_ld + h * p.vdim + v] = from_f<T>(__int_as_float(0x7fc00000));
            continue;
        }
        const T* kseq = static_cast<const T*>(p.k) + block * p.k_seq + g * p.k_head;
        const T* vseq = static_cast<const T*>(p.v) + block * p.v_seq + g * p.v_head;
        const T* kr_seq = static_cast<const T*>(p.krot) + (int64_t)b * p.rows_per_seq * p.krot_ld;
        float m = -INFINITY, l = 0.f, acc[AW_MAXV];
#pragma unroll
        for (int v = 0; v < AW_MAXV; ++v) acc[v] = 0.f;
        for (int k0 = first; k0 <= last; k0 += 32) {
            const int k = k0 + lane;
            float sc = -INFINITY;
            if (k <= last) {
                const T* kn = kseq + k * p.k_ld;
                const T* kr = kr_seq + k * p.krot_ld;
                float d = 0.f;
                for (int e = 0; e < p.dim; ++e) d = fmaf(qs[e], to_f(kn[e]), d);
                for (int e = 0; e < p.rot; ++e) d = fmaf(qs[p.dim + e], to_f(kr[e]), d);
                sc = d * scale;
            }
            float mx = sc;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m_new = fmaxf(m, mx);
            const float shrink = expf(m - m_new);      // 0 at the first keys (m = -inf)
            const float w = expf(sc - m_new);
            float sum = w;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l = l * shrink + sum;
            m = m_new;
#pragma unroll
            for (int v = 0; v < AW_MAXV; ++v) acc[v] *= shrink;
            const int nk = min(32, last - k0 + 1);
            for (int j = 0; j < nk; ++j) {
                const float wj = __shfl_sync(0xffffffffu, w, j);
                const T* vr = vseq + (k0 + j) * p.v_ld;
#pragma unroll
                for (int v = 0; v < AW_MAXV; ++v)
                    if (v * 32 + lane < p.vdim) acc[v] = fmaf(wj, to_f(vr[v * 32 + lane]), acc[v]);
            }
        }
        T* out = static_cast<T*>(p.out) + row * p.out_ld + h * p.vdim;
#pragma unroll
        for (int v = 0; v < AW_MAXV; ++v)
            if (v * 32 + lane < p.vdim) {
                float o = acc[v] / l;
                if (p.gate) o *= sigmoid_exact(to_f(static_cast<const T*>(p.gate)[row * p.gate_ld + h * p.vdim + v * 32 + lane]));
                out[v * 32 + lane] = from_f<T>(o);
            }
        if (h == p.H - 1)                                   // the padding columns behind the last head
            for (int i = p.H * p.vdim + lane; i < p.out_ld; i += 32)
                static_cast<T*>(p.out)[row * p.out_ld + i] = from_f<T>(0.f);
    }
}

int attn_any(const AttnPortionParams& p, int dtype, cudaStream_t st, const char* what) {
    if (p.vdim > AW_MAXV * 32) return fail(BN_ERR_UNSUPPORTED, "%s: vdim=%d (at most %d)", what, p.vdim, AW_MAXV * 32);
    const size_t smem = (size_t)AW_WARPS * (p.dim + p.rot) * sizeof(float);
    const long long blocks = ((long long)p.B * p.S * p.H + AW_WARPS - 1) / AW_WARPS, cap = (long long)sm_count() * 64;
    const unsigned grid = (unsigned)(blocks < cap ? blocks : cap);
    if (dtype == 0) {
        if (int rc = allow_smem(attn_any_kernel<float>, smem, what)) return rc;
        launch_dependent(attn_any_kernel<float>, grid, AW_WARPS * 32, smem, st, p);
    } else {
        if (int rc = allow_smem(attn_any_kernel<__nv_bfloat16>, smem, what)) return rc;
        launch_dependent(attn_any_kernel<__nv_bfloat16>, grid, AW_WARPS * 32, smem, st, p);
    }
    return launch_status(what);
}

}  // namespace bn

using namespace bn;

extern "C" int bn_attn_window(const void* q, int64_t q_ld, const void* k, const void* v, int64_t kv_ld, const void* krot,
                              int64_t krot_ld, void* out, int64_t out_ld, int B, int S, int n_old, int rows_per_seq, int H,
                              int dim, int rot, int vdim, int window, float scale, int* error_word, int dtype,
                              bn_stream_t stream) {
    const char* what = "bn_attn_window";
    if (!q || !k || !v || !krot || !out) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || S < 0 || n_old < 0 || n_old + S > rows_per_seq || H <= 0 || dim <= 0 || rot < 0 || vdim <= 0 || window <= 0 || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d S=%d n_old=%d H=%d dim=%d rot=%d vdim=%d window=%d", what, B, S, n_old,
                    H, dim, rot, vdim, window);
    if (int rc = require_sm100()) return rc;
    if (B == 0 || S == 0) return BN_OK;
    AttnPortionParams p{};
    p.q = q; p.k = k; p.v = v; p.krot = krot; p.out = out;
    p.q_ld = q_ld; p.k_ld = p.v_ld = kv_ld; p.krot_ld = krot_ld; p.out_ld = out_ld;
    p.k_head = dim; p.v_head = vdim; p.k_seq = p.v_seq = rows_per_seq * kv_ld;
    p.B = B; p.S = S; p.n_old = n_old; p.rows_per_seq = rows_per_seq; p.H = p.kv_heads = H; p.dim = dim; p.rot = rot; p.vdim = vdim;
    p.mask = MASK_WINDOW; p.span = window; p.scale = scale; p.error_word = error_word;
    if (dtype == 1 && attn_portion_sm100_ok(p)) return attn_portion_sm100(p, as_stream(stream));
    return attn_any(p, dtype, as_stream(stream), what);
}

extern "C" int bn_attn_chunked(const void* q, int64_t q_ld, const void* k, int64_t k_ld, const void* v, int64_t v_ld,
                               const void* gate, int64_t gate_ld, void* out, int64_t out_ld, int B, int S, int n_old,
                               int rows_per_seq, int H, int kv_heads, int dim, int vdim, int chunk, int rms_dim, float rms_eps,
                               float scale, float score_bound, int* error_word, int dtype, bn_stream_t stream) {
    const char* what = "bn_attn_chunked";
    if (!q || !k || !v || !out) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || S < 0 || n_old < 0 || n_old >= chunk || n_old + S > rows_per_seq || H <= 0 || kv_heads <= 0 || H % kv_heads || dim <= 0 ||
        vdim <= 0 || rms_dim < 0 || rms_dim > dim || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d S=%d n_old=%d H=%d kv_heads=%d dim=%d vdim=%d chunk=%d", what, B, S, n_old, H,
                    kv_heads, dim, vdim, chunk);
    if (int rc = require_sm100()) return rc;
    if (B == 0 || S == 0) return BN_OK;
    AttnPortionParams p{};
    p.q = q; p.k = k; p.v = v; p.gate = gate; p.out = out;
    p.q_ld = q_ld; p.k_ld = k_ld; p.v_ld = v_ld; p.gate_ld = gate_ld; p.out_ld = out_ld;
    p.k_head = dim; p.v_head = vdim; p.k_seq = rows_per_seq * k_ld; p.v_seq = rows_per_seq * v_ld;
    p.B = B; p.S = S; p.n_old = n_old; p.rows_per_seq = rows_per_seq; p.H = H; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim;
    p.mask = MASK_CHUNK; p.span = chunk; p.rms_dim = rms_dim; p.rms_eps = rms_eps; p.scale = scale; p.score_bound = score_bound;
    p.error_word = error_word;
    if (dtype == 1 && attn_portion_sm100_ok(p)) return attn_portion_sm100(p, as_stream(stream));
    return attn_any(p, dtype, as_stream(stream), what);
}
