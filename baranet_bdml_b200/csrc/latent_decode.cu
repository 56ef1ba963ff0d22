// One-token latent attention on warp-level tensor cores (bf16): scores of up to 16 heads against the cached latents and
// the weighted latent sum, from ONE read of the cache.
//
// All heads share the cached row [latent | rotated key part], so the heads are the M = 16 of mma.sync.m16n8k16 and the
// kernel is a stream of the ring through the SMs: about 2 * 16 * (2 kv_rank + rot) FLOP per row of 2 (kv_rank + rot) bytes.
// (tcgen05's smallest M is 64: three quarters of each instruction would be padding.)
//
// CTA = (row, group of 16 heads, split) with nine warps: warp 8 streams tiles of 64 ring rows by TMA (64-column blocks,
// 128-byte swizzle, ring of stages); warps 0-7 compute, per tile:
//   scores   warp w: ring rows 16 (w % 4) .. + 15, half w / 4 of the columns; the halves are added in shared memory
//   softmax  warp w: heads 2 w, 2 w + 1; half a warp per head; running maximum
//   sum      warp w: an eighth of the latent's columns, all 64 rows
// Softmax does not care about order, so the ring is walked in ROW order: row r holds position pos - (pos - r mod ring),
// and a row whose position is outside the window (or was never written) gets weight zero.
// A split's result is its normalised sum and log-sum-exp; bn_latent_expand_out merges the splits (in place).
// Waits are bounded: on expiry the CTA stops and leaves a NaN log-sum-exp, which surfaces as NaN logits.
#include "common.cuh"
#include "hybrid.cuh"
#include "latent.cuh"
#include "ptx.cuh"
#include "tma.cuh"

namespace bn {

using namespace ptx;

constexpr int LM_ROWS = 64, LM_BLK = LM_ROWS * 128;     // a 64-column block of a tile: 8 KB
constexpr int LM_THREADS = 288;
constexpr int LM_MAXSTAGE = 6;
constexpr int LM_SMEM_LIMIT = 226 * 1024;
constexpr int LM_NT = 8;                                // 8-column pieces of the latent per warp: kv_ld <= 512
constexpr float LM_LOG2E = 1.4426950408889634f, LM_LN2 = 0.6931471805599453f;

struct LmLayout {
    int nblk, stages;
    size_t q, s, pw, alpha, tiles, total;               // byte offsets
};

__host__ __device__ inline LmLayout lm_layout(int kv_ld, int rot_ld) {
    LmLayout L;
    const int width = kv_ld + rot_ld;
    L.nblk = (width + 63) / 64;
    const int q_ld = L.nblk * 64 + 8;
    L.q = 0;                                            // [16][q_ld] bf16
    L.s = L.q + (size_t)16 * q_ld * 2;                  // [2][16][LM_ROWS + 4] fp32
    L.pw = L.s + (size_t)2 * 16 * (LM_ROWS + 4) * 4;    // [16][LM_ROWS + 8] bf16
    L.alpha = L.pw + (size_t)16 * (LM_ROWS + 8) * 2;    // [16] fp32
    L.tiles = (L.alpha + 64 + 1023) / 1024 * 1024;
    const size_t stage = (size_t)L.nblk * LM_BLK;
    long long left = (long long)LM_SMEM_LIMIT - 1024 - (long long)L.tiles;
    int n = left > 0 ? (int)(left / (long long)stage) : 0;
    L.stages = n > LM_MAXSTAGE ? LM_MAXSTAGE : n;
    L.total = 1024 + L.tiles + (size_t)L.stages * stage;
    return L;
}

struct LmParams {
    const __nv_bfloat16* q_abs;
    const int32_t *seq_ids, *positions;
    float *partial, *lse;
    int B, H, kv_ld, rot_ld, ring_tokens, window, splits, groups;
    float scale_log2;
};

__global__ void __launch_bounds__(LM_THREADS, 1)
latent_decode_mma_kernel(const __grid_constant__ CUtensorMap tmap, const LmParams p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t bar_full[LM_MAXSTAGE], bar_empty[LM_MAXSTAGE];
    __shared__ int s_abort;
    const int tid = threadIdx.x, warp = tid / 32, lane = tid % 32;
    const LmLayout L = lm_layout(p.kv_ld, p.rot_ld);
    uint8_t* base = smem_raw + (((smem_u32(smem_raw) + 1023u) & ~1023u) - smem_u32(smem_raw));
    const uint32_t base_u = smem_u32(base);
    const int width = p.kv_ld + p.rot_ld, q_ld = L.nblk * 64 + 8;
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(base + L.q);
    float* ss = reinterpret_cast<float*>(base + L.s);
    __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(base + L.pw);
    float* salpha = reinterpret_cast<float*>(base + L.alpha);
    const uint32_t sT = base_u + (uint32_t)L.tiles;
    const int split = blockIdx.x % p.splits, grp = (blockIdx.x / p.splits) % p.groups, b = blockIdx.x / (p.splits * p.groups);
    const int h0 = grp * 16, nh = min(16, p.H - h0);

    if (tid == 0) {
        for (int s = 0; s < LM_MAXSTAGE; ++s) {
            mbar_init(smem_u32(&bar_full[s]), 1);
            mbar_init(smem_u32(&bar_empty[s]), 8);
        }
        s_abort = 0;
        fence_mbar_init();
        prefetch_tensormap(&tmap);
    }
    grid_dependency_wait();
    grid_launch_dependents();
    const int pos = p.positions[b], slot = p.seq_ids ? p.seq_ids[b] : b;
    const int used = min(pos + 1, p.ring_tokens);               // ring rows written so far
    const int n_tiles = (used + LM_ROWS - 1) / LM_ROWS;
    const int per = (n_tiles + p.splits - 1) / p.splits;
    const int t_begin = min(n_tiles, split * per), t_end = min(n_tiles, t_begin + per);
    // queries of the group, zeros beyond its heads and its columns
    for (int i = tid; i < 16 * (q_ld / 8); i += LM_THREADS) {
        const int h = i / (q_ld / 8), c = (i - h * (q_ld / 8)) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (h < nh && c < width) v = *reinterpret_cast<const uint4*>(p.q_abs + ((int64_t)b * p.H + h0 + h) * width + c);
        *reinterpret_cast<uint4*>(sq + h * q_ld + c) = v;
    }
    __syncthreads();

    const int64_t part0 = ((int64_t)b * p.H + h0) * p.splits + split;       // + head * splits
    if (warp == 8) {
        if (lane == 0) {
            const uint64_t policy = l2_policy_evict_first();
            for (int t = t_begin, it = 0; t < t_end; ++t, ++it) {
                const int stage = it % L.stages;
                if (!mbar_wait(smem_u32(&bar_empty[stage]), ((it / L.stages) & 1u) ^ 1u, &s_abort)) break;
                mbar_arrive_expect_tx(smem_u32(&bar_full[stage]), L.nblk * LM_BLK);
                for (int x = 0; x < L.nblk; ++x)
                    tma_load_2d_hint(sT + (stage * L.nblk + x) * LM_BLK, &tmap, x * 64, slot * p.ring_tokens + t * LM_ROWS,
                                     smem_u32(&bar_full[stage]), policy);
            }
        }
        return;
    }

    const int g = lane / 4, j = lane % 4;
    const int k_steps = (width + 15) / 16, k_half = (k_steps + 1) / 2;
    const int rg = warp % 4, half = warp / 4;
    const int ks0 = half * k_half, ks1 = min(k_steps, ks0 + k_half);
    const int n_pieces = p.kv_ld / 8, per_warp = (n_pieces + 7) / 8;        // 8-column pieces of the latent
    const int pc0 = warp * per_warp, npc = max(0, min(per_warp, n_pieces - pc0));
    float acc[LM_NT][4];
#pragma unroll
    for (int i = 0; i < LM_NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const int sh = 2 * warp + lane / 16, sc = (lane % 16) * 4;              // softmax: this lane's head and first column
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int t = t_begin, it = 0; t < t_end; ++t, ++it) {
        const int stage = it % L.stages;
        ok = mbar_wait(smem_u32(&bar_full[stage]), (it / L.stages) & 1u, &s_abort);
        // all eight warps leave together: the named barrier ORs the verdict
        if (named_bar_or(1, 256, !ok)) { ok = false; break; }
        const uint32_t tile = sT + stage * L.nblk * LM_BLK;
        // ---- scores: 16 heads x 16 rows over this warp's half of the columns
        {
            float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
            const int row = rg * 16 + (lane / 16) * 8 + lane % 8;           // B fragments: matrices (rows 0-7 | 8-15) x (k 0-7 | 8-15)
            const int kpart = (lane / 8) % 2;
            const uint32_t qa = base_u + (uint32_t)L.q + ((lane % 16) * q_ld + (lane / 16) * 8) * 2;
#pragma unroll 4
            for (int ks = ks0; ks < ks1; ++ks) {
                uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
                ldmatrix_x4(qa + ks * 32, a0, a1, a2, a3);
                const int chunk = ks * 2 + kpart;
                ldmatrix_x4(tile + (chunk / 8) * LM_BLK + row * 128 + (((chunk % 8) ^ (row & 7)) << 4), b0, b1, b2, b3);
                mma_bf16_16816(c0, a0, a1, a2, a3, b0, b1);
                mma_bf16_16816(c1, a0, a1, a2, a3, b2, b3);
            }
            float* d = ss + (half * 16) * (LM_ROWS + 4) + rg * 16 + 2 * j;
            *reinterpret_cast<float2*>(d + g * (LM_ROWS + 4)) = make_float2(c0[0], c0[1]);
            *reinterpret_cast<float2*>(d + (g + 8) * (LM_ROWS + 4)) = make_float2(c0[2], c0[3]);
            *reinterpret_cast<float2*>(d + g * (LM_ROWS + 4) + 8) = make_float2(c1[0], c1[1]);
            *reinterpret_cast<float2*>(d + (g + 8) * (LM_ROWS + 4) + 8) = make_float2(c1[2], c1[3]);
        }
        named_bar_sync(2, 256);
        // ---- softmax of two heads per warp
        {
            const float4 u = *reinterpret_cast<const float4*>(ss + sh * (LM_ROWS + 4) + sc);
            const float4 v = *reinterpret_cast<const float4*>(ss + (16 + sh) * (LM_ROWS + 4) + sc);
            float s[4] = {u.x + v.x, u.y + v.y, u.z + v.z, u.w + v.w};
            float mx = -INFINITY;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = t * LM_ROWS + sc + e;
                int back = (pos - r) % p.ring_tokens;                       // how far back the row's token lies
                if (back < 0) back += p.ring_tokens;
                const bool seen = r < used && back < p.window;
                s[e] = seen ? s[e] * p.scale_log2 : -INFINITY;
                mx = fmaxf(mx, s[e]);
            }
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m_new = fmaxf(m_run, mx);
            const float ref = m_new == -INFINITY ? 0.f : m_new;
            const float alpha = m_run == -INFINITY ? 0.f : ex2(m_run - ref);
            float sum = 0.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) { s[e] = ex2(s[e] - ref); sum += s[e]; }
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l_run = fmaf(l_run, alpha, sum);
            m_run = m_new;
            *reinterpret_cast<uint2*>(sp + sh * (LM_ROWS + 8) + sc) = make_uint2(pack_bf16(s[0], s[1]), pack_bf16(s[2], s[3]));
            if (lane % 16 == 0) salpha[sh] = alpha;
        }
        named_bar_sync(1, 256);
        // ---- weighted sum over this warp's columns
        if (npc > 0) {
            const float al = salpha[g], ah = salpha[g + 8];
#pragma unroll
            for (int i = 0; i < LM_NT; ++i) { acc[i][0] *= al; acc[i][1] *= al; acc[i][2] *= ah; acc[i][3] *= ah; }
            const uint32_t pa = base_u + (uint32_t)L.pw + ((lane % 16) * (LM_ROWS + 8) + (lane / 16) * 8) * 2;
            uint32_t a[4][4];
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) ldmatrix_x4(pa + ks * 32, a[ks][0], a[ks][1], a[ks][2], a[ks][3]);
#pragma unroll
            for (int i = 0; i < LM_NT; ++i) {
                if (i >= npc) break;
                const int chunk = pc0 + i;
                const uint32_t blk = tile + (chunk / 8) * LM_BLK + (((chunk % 8) ^ (lane & 7)) << 4);
#pragma unroll
                for (int kp = 0; kp < 2; ++kp) {                            // 32 rows per load: four 8 x 8 matrices, transposed
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4_trans(blk + (kp * 32 + lane) * 128, b0, b1, b2, b3);
                    mma_bf16_16816(acc[i], a[2 * kp][0], a[2 * kp][1], a[2 * kp][2], a[2 * kp][3], b0, b1);
                    mma_bf16_16816(acc[i], a[2 * kp + 1][0], a[2 * kp + 1][1], a[2 * kp + 1][2], a[2 * kp + 1][3], b2, b3);
                }
            }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(&bar_empty[stage]));
    }
    // ---- the split's result
    named_bar_sync(1, 256);                                    // salpha may still be read
    if (lane % 16 == 0) {
        if (sh < nh)
            p.lse[part0 + (int64_t)sh * p.splits] = !ok ? __int_as_float(0x7fc00000) : l_run > 0.f ? (m_run + log2f(l_run)) * LM_LN2 : -INFINITY;
        salpha[sh] = l_run > 0.f ? 1.f / l_run : 0.f;
    }
    named_bar_sync(2, 256);
    const float il = salpha[g], ih = salpha[g + 8];
#pragma unroll
    for (int i = 0; i < LM_NT; ++i) {
        if (i >= npc) break;
        const int col = (pc0 + i) * 8 + 2 * j;
        if (g < nh)
            *reinterpret_cast<float2*>(p.partial + (part0 + (int64_t)g * p.splits) * p.kv_ld + col) = make_float2(acc[i][0] * il, acc[i][1] * il);
        if (g + 8 < nh)
            *reinterpret_cast<float2*>(p.partial + (part0 + (int64_t)(g + 8) * p.splits) * p.kv_ld + col) =
                make_float2(acc[i][2] * ih, acc[i][3] * ih);
    }
}

bool latent_decode_mma_ok(int H, int kv_ld, int rot_ld) {
    return H > 0 && kv_ld <= LM_NT * 8 * 8 && lm_layout(kv_ld, rot_ld).stages >= 2;
}

// One CTA runs per SM: choose the cut of the window whose waves of CTAs take the least time, a CTA costing its tiles plus
// about one and a half for its start and its end.
int latent_decode_mma_splits(int B, int H, int window, int sms) {
    const int tiles = (window + LM_ROWS - 1) / LM_ROWS;
    const long long items = (long long)B * ((H + 15) / 16);
    int best = 1;
    double best_cost = 1e30;
    for (int s = 1; s <= tiles && s <= 64; ++s) {
        const long long waves = (items * s + sms - 1) / sms;
        const double cost = (double)waves * ((tiles + s - 1) / s + 1.5) + 0.02 * s;
        if (cost < best_cost) { best_cost = cost; best = s; }
    }
    return best;
}

int latent_decode_mma(const LatentDecodeParams& a, cudaStream_t st) {
    const char* what = "bn_latent_decode";
    const int width = a.kv_ld + a.rot_ld;
    if ((reinterpret_cast<uintptr_t>(a.q_abs) | reinterpret_cast<uintptr_t>(a.ring) | reinterpret_cast<uintptr_t>(a.partial)) & 15)
        return fail(BN_ERR_INVALID_ARG, "%s: q_abs, ring and partial must be 16-byte aligned", what);
    // the last tile of a slot may reach into the next slot's rows (they get weight zero), never behind the last slot
    CUtensorMap tmap;
    {
        const uint64_t dims[2] = {(uint64_t)width, (uint64_t)a.num_slots * a.ring_tokens}, strides[1] = {(uint64_t)width * 2};
        const uint32_t box[2] = {64, LM_ROWS};
        if (int rc = make_tensor_map(&tmap, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.ring, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B))
            return rc;
    }
    const LmLayout L = lm_layout(a.kv_ld, a.rot_ld);
    LmParams p{static_cast<const __nv_bfloat16*>(a.q_abs), a.seq_ids, a.positions, a.partial, a.lse, a.B, a.H, a.kv_ld, a.rot_ld,
               a.ring_tokens, a.window, a.splits, (a.H + 15) / 16, a.scale * LM_LOG2E};
    int dev = 0;
    cudaGetDevice(&dev);
    static thread_local int configured_dev = -1;
    if (configured_dev != dev) {
        cudaError_t e = cudaFuncSetAttribute(latent_decode_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LM_SMEM_LIMIT);
        if (e != cudaSuccess) return fail(BN_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
        configured_dev = dev;
    }
    launch_dependent(latent_decode_mma_kernel, (unsigned)((long long)a.B * p.groups * a.splits), LM_THREADS, L.total, st, tmap, p);
    return launch_status(what);
}

// ---------------------------------------------------------------------------------------------------------------
// The two per-head products around it.  Both stream a head's weight once per 16 rows and request it before they wait for
// the launch ahead of them: weights depend on nothing.
// ---------------------------------------------------------------------------------------------------------------
struct AbsorbParams {
    const __nv_bfloat16 *q, *wuk;
    const double* freq;
    const int32_t* positions;
    __nv_bfloat16* q_abs;
    int64_t q_ld;
    int B, H, dim, rot, kv_ld, rot_ld, kp, n_tiles;      // kp: dim rounded up to 16
    int vec;                                             // query rows and heads start on 16-byte boundaries
};

constexpr int AB_N = 64;

// q_abs = q W_uk for 16 rows, one head, 64 latent columns; the last tile of a head is its rotated part
__global__ void __launch_bounds__(128)
latent_absorb_mma_kernel(const AbsorbParams p) {
    extern __shared__ __align__(16) uint8_t smem[];
    const int lda = p.kp + 8;
    __nv_bfloat16* sw = reinterpret_cast<__nv_bfloat16*>(smem);          // [kp][AB_N + 8]
    __nv_bfloat16* sa = sw + p.kp * (AB_N + 8);                          // [16][kp + 8]
    const int tile = blockIdx.x % (p.n_tiles + 1), h = blockIdx.x / (p.n_tiles + 1) % p.H;
    const int b0 = blockIdx.x / ((p.n_tiles + 1) * p.H) * 16, nb = min(16, p.B - b0);
    const int width = p.kv_ld + p.rot_ld, E = p.dim + p.rot, n0 = tile * AB_N;
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    if (tile < p.n_tiles) {
        const __nv_bfloat16* w = p.wuk + (int64_t)h * p.dim * p.kv_ld + n0;
        for (int i = threadIdx.x; i < p.kp * (AB_N / 8); i += 128) {
            const int k = i / (AB_N / 8), c = i % (AB_N / 8) * 8;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (k < p.dim && n0 + c < p.kv_ld) v = __ldg(reinterpret_cast<const uint4*>(w + (int64_t)k * p.kv_ld + c));
            *reinterpret_cast<uint4*>(sw + k * (AB_N + 8) + c) = v;
        }
    }
    grid_dependency_wait();
    grid_launch_dependents();
    const __nv_bfloat16* q = p.q + (int64_t)b0 * p.q_ld + h * E;
    if (tile == p.n_tiles) {
        for (int i = threadIdx.x; i < nb * (p.rot_ld / 2); i += 128) {
            const int b = i / (p.rot_ld / 2), j = i % (p.rot_ld / 2);
            uint32_t o = 0;
            if (2 * j < p.rot) {
                const __nv_bfloat16* x = q + b * p.q_ld + p.dim + 2 * j;
                const float u = to_f(x[0]), v = to_f(x[1]);
                float cs, sn;
                rotation(p.positions[b0 + b], p.freq[j], &cs, &sn);
                o = pack_bf16(u * cs - v * sn, v * cs + u * sn);
            }
            *reinterpret_cast<uint32_t*>(p.q_abs + ((int64_t)(b0 + b) * p.H + h) * width + p.kv_ld + 2 * j) = o;
        }
        return;
    }
    if (p.vec) {
        for (int i = threadIdx.x; i < 16 * (p.kp / 8); i += 128) {
            const int b = i / (p.kp / 8), c = i % (p.kp / 8) * 8;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (b < nb && c < p.dim) v = *reinterpret_cast<const uint4*>(q + b * p.q_ld + c);
            *reinterpret_cast<uint4*>(sa + b * lda + c) = v;
        }
    } else {
        for (int i = threadIdx.x; i < 16 * p.kp; i += 128) {
            const int b = i / p.kp, c = i % p.kp;
            sa[b * lda + c] = b < nb && c < p.dim ? q[b * p.q_ld + c] : __float2bfloat16(0.f);
        }
    }
    __syncthreads();
    float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t ua = smem_u32(sa) + ((lane % 16) * lda + (lane / 16) * 8) * 2;
    const uint32_t uw = smem_u32(sw) + ((lane % 16) * (AB_N + 8) + warp * 16 + (lane / 16) * 8) * 2;
#pragma unroll 4
    for (int ks = 0; ks < p.kp / 16; ++ks) {
        uint32_t a0, a1, a2, a3, w0, w1, w2, w3;
        ldmatrix_x4(ua + ks * 32, a0, a1, a2, a3);
        ldmatrix_x4_trans(uw + ks * 16 * (AB_N + 8) * 2, w0, w1, w2, w3);
        mma_bf16_16816(c0, a0, a1, a2, a3, w0, w1);
        mma_bf16_16816(c1, a0, a1, a2, a3, w2, w3);
    }
    const int g = lane / 4, j = lane % 4;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int b = g + 8 * r;
        if (b >= nb) continue;
        __nv_bfloat16* o = p.q_abs + ((int64_t)(b0 + b) * p.H + h) * width + n0 + warp * 16 + 2 * j;
        if (n0 + warp * 16 + 2 * j < p.kv_ld) *reinterpret_cast<uint32_t*>(o) = pack_bf16(c0[2 * r], c0[2 * r + 1]);
        if (n0 + warp * 16 + 8 + 2 * j < p.kv_ld) *reinterpret_cast<uint32_t*>(o + 8) = pack_bf16(c1[2 * r], c1[2 * r + 1]);
    }
}

bool latent_absorb_mma(const void* q, int64_t q_ld, const void* wuk, const double* freq, const int32_t* positions, void* q_abs, int B,
                       int H, int dim, int rot, int kv_ld, int rot_ld, cudaStream_t st) {
    const int kp = (dim + 15) / 16 * 16;
    const size_t smem = ((size_t)kp * (AB_N + 8) + 16 * (kp + 8)) * 2;
    if (smem > 48 * 1024 || (reinterpret_cast<uintptr_t>(wuk) & 15) || (reinterpret_cast<uintptr_t>(q_abs) & 3)) return false;
    AbsorbParams p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(wuk), freq, positions,
                   static_cast<__nv_bfloat16*>(q_abs), q_ld, B, H, dim, rot, kv_ld, rot_ld, kp, (kv_ld + AB_N - 1) / AB_N, 0};
    p.vec = dim % 8 == 0 && rot % 8 == 0 && q_ld % 8 == 0 && (reinterpret_cast<uintptr_t>(q) & 15) == 0;
    launch_dependent(latent_absorb_mma_kernel, (unsigned)((p.n_tiles + 1) * H * ((B + 15) / 16)), 128, smem, st, p);
    return true;
}

// Merges a (row, head)'s splits into its split 0: a thread owns four columns of all splits, which it reads before it writes.
constexpr int MG_MAXSPLITS = 64, MG_BATCH = 8;

__global__ void __launch_bounds__(128)
latent_merge_kernel(float* partial, const float* lse, int splits, int kv_ld) {
    __shared__ float s_w[MG_MAXSPLITS];
    grid_dependency_wait();
    grid_launch_dependents();
    float* base = partial + (int64_t)blockIdx.x * splits * kv_ld;
    float4 f[MG_BATCH];
    const int c0 = threadIdx.x * 4;
    if (c0 < kv_ld) {
#pragma unroll
        for (int s = 0; s < MG_BATCH; ++s)
            if (s < splits) f[s] = *reinterpret_cast<const float4*>(base + (int64_t)s * kv_ld + c0);
    }
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        const float* l = lse + (int64_t)blockIdx.x * splits;
        const float x0 = lane < splits ? l[lane] : -INFINITY, x1 = lane + 32 < splits ? l[lane + 32] : -INFINITY;
        float m = fmaxf(x0, x1);                 // drops a NaN (a split that gave up); the sum below keeps it
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        const float e0 = m == -INFINITY ? 0.f : expf(x0 - m), e1 = m == -INFINITY ? 0.f : expf(x1 - m);
        float t = e0 + e1;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
        const float inv = t == 0.f ? 0.f : 1.f / t;
        if (lane < splits) s_w[lane] = e0 * inv;
        if (lane + 32 < splits) s_w[lane + 32] = e1 * inv;
    }
    __syncthreads();
    for (int c = c0; c < kv_ld; c += 512) {
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s0 = 0; s0 < splits; s0 += MG_BATCH) {
            if (c > c0 || s0 > 0) {
#pragma unroll
                for (int s = 0; s < MG_BATCH; ++s)
                    if (s0 + s < splits) f[s] = *reinterpret_cast<const float4*>(base + (int64_t)(s0 + s) * kv_ld + c);
            }
#pragma unroll
            for (int s = 0; s < MG_BATCH; ++s)
                if (s0 + s < splits) {
                    const float x = s_w[s0 + s];
                    o.x = fmaf(f[s].x, x, o.x);
                    o.y = fmaf(f[s].y, x, o.y);
                    o.z = fmaf(f[s].z, x, o.z);
                    o.w = fmaf(f[s].w, x, o.w);
                }
        }
        *reinterpret_cast<float4*>(base + c) = o;
    }
}

struct ExpandParams {
    const float *sums, *lse;                             // sums: [B][H], `stride` floats apart
    const __nv_bfloat16* wuv;
    __nv_bfloat16* out;
    int64_t out_ld, stride;
    int B, H, vdim, kv_ld, v_tiles, steps;               // steps: 32-wide pieces of the latent, rounded up
};

constexpr int EX_V = 32, EX_BATCH = 8;

// out = o W_uv^T for 16 rows, one head, 32 value columns.  Eight warps = 4 pieces of 8 columns x 2 halves of the latent.  A
// lane holds 16 contiguous bytes of a weight row per 32-wide step and takes the same columns of two rows of the sums from
// shared memory: any order of the inner index serves, as long as both sides use it.  `lse` (an unmerged single split) is
// looked at only for the mark of a split that gave up.
__global__ void __launch_bounds__(256)
latent_expand_mma_kernel(const ExpandParams p) {
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ float s_part[8][16][9];
    __nv_bfloat16* so = reinterpret_cast<__nv_bfloat16*>(smem);          // [16][steps * 32 + 8]
    const int ldo = p.steps * 32 + 8;
    const int vt = blockIdx.x % p.v_tiles, h = blockIdx.x / p.v_tiles % p.H;
    const int b0 = blockIdx.x / (p.v_tiles * p.H) * 16, nb = min(16, p.B - b0);
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, g = lane / 4, j = lane % 4;
    const int half = (p.steps + 1) / 2, s0 = warp / 4 * half, s1 = min(p.steps, s0 + half);
    const int v = vt * EX_V + warp % 4 * 8 + g;
    const __nv_bfloat16* w = p.wuv + ((int64_t)h * p.vdim + v) * p.kv_ld + j * 8;
    uint4 wv[EX_BATCH];
    auto load_w = [&](int s) {
#pragma unroll
        for (int i = 0; i < EX_BATCH; ++i) {
            wv[i] = make_uint4(0, 0, 0, 0);
            if (s + i < s1 && v < p.vdim && (s + i) * 32 + j * 8 < p.kv_ld) wv[i] = __ldg(reinterpret_cast<const uint4*>(w + (s + i) * 32));
        }
    };
    load_w(s0);
    grid_dependency_wait();
    grid_launch_dependents();
    const int pieces = p.steps * 8;                                       // of 4 columns
#pragma unroll 8
    for (int i = threadIdx.x; i < 16 * pieces; i += 256) {
        const int b = i / pieces, c = i % pieces * 4;
        float x[4] = {0.f, 0.f, 0.f, 0.f};
        if (b < nb && c < p.kv_ld) load4(p.sums + ((int64_t)(b0 + b) * p.H + h) * p.stride + c, x);
        store4(so + b * ldo + c, x);
    }
    __syncthreads();
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int s = s0; s < s1; s += EX_BATCH) {
        if (s > s0) load_w(s);
#pragma unroll
        for (int i = 0; i < EX_BATCH; ++i) {
            if (s + i >= s1) break;
            const uint4 lo = *reinterpret_cast<const uint4*>(so + g * ldo + (s + i) * 32 + j * 8);
            const uint4 hi = *reinterpret_cast<const uint4*>(so + (g + 8) * ldo + (s + i) * 32 + j * 8);
            mma_bf16_16816(acc, lo.x, hi.x, lo.y, hi.y, wv[i].x, wv[i].y);
            mma_bf16_16816(acc, lo.z, hi.z, lo.w, hi.w, wv[i].z, wv[i].w);
        }
    }
    s_part[warp][g][2 * j] = acc[0];
    s_part[warp][g][2 * j + 1] = acc[1];
    s_part[warp][g + 8][2 * j] = acc[2];
    s_part[warp][g + 8][2 * j + 1] = acc[3];
    __syncthreads();
    for (int i = threadIdx.x; i < 16 * EX_V; i += 256) {
        const int b = i / EX_V, c = i % EX_V, col = vt * EX_V + c;
        if (b < nb && col < p.vdim) {
            float y = s_part[c / 8][b][c % 8] + s_part[4 + c / 8][b][c % 8];
            if (p.lse) {
                const float l = p.lse[(int64_t)(b0 + b) * p.H + h];
                if (l != l) y = l;
            }
            p.out[(b0 + b) * p.out_ld + h * p.vdim + col] = __float2bfloat16(y);
        }
    }
    if (h == p.H - 1 && vt == 0)                                          // the padding columns behind the last head
        for (int b = 0; b < nb; ++b)
            for (int i = p.H * p.vdim + threadIdx.x; i < p.out_ld; i += 256) p.out[(b0 + b) * p.out_ld + i] = __float2bfloat16(0.f);
}

bool latent_expand_mma(float* partial, const float* lse, int splits, const void* wuv, void* out, int64_t out_ld, int B, int H,
                       int vdim, int kv_ld, cudaStream_t st) {
    const int steps = (kv_ld + 31) / 32;
    const size_t smem = (size_t)16 * (steps * 32 + 8) * 2;
    if (splits > MG_MAXSPLITS || smem > 32 * 1024 || ((reinterpret_cast<uintptr_t>(wuv) | reinterpret_cast<uintptr_t>(partial)) & 15)) return false;
    if (splits > 1) launch_dependent(latent_merge_kernel, (unsigned)(B * H), 128, 0, st, partial, lse, splits, kv_ld);
    ExpandParams p{partial, splits > 1 ? nullptr : lse, static_cast<const __nv_bfloat16*>(wuv), static_cast<__nv_bfloat16*>(out), out_ld,
                   (int64_t)splits * kv_ld, B, H, vdim, kv_ld, (vdim + EX_V - 1) / EX_V, steps};
    launch_dependent(latent_expand_mma_kernel, (unsigned)(p.v_tiles * H * ((B + 15) / 16)), 256, smem, st, p);
    return true;
}

}  // namespace bn
