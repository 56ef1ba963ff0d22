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
// A split's result is its normalised sum and log-sum-exp; bn_latent_expand_out merges the splits.
// Waits are bounded: on expiry the CTA stops and leaves a NaN log-sum-exp, which surfaces as NaN logits.
#include "common.cuh"
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

}  // namespace bn
