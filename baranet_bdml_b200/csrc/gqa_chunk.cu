// Grouped-query attention in chunks of positions: what lies between the q/k/v/gate projection and the output projection
// apart from the portion attention itself.
//
//   keys        divided by their root mean square per head (in the cache they are already)
//   values      optionally (1 - lambda) v + lambda v_first, v_first an earlier layer's values of the same token
//   queries     divided by their root mean square through the score scale
//   a position sees the keys of its own chunk up to its own, chunks counted from position 0
//   the result  optionally multiplied by the sigmoid of a gate
//
// Cache: ring_k[slot][kv_head][ring_tokens][dim_ld] and ring_v likewise, the token of position p in row p % chunk; a chunk
// overwrites the one before it.  ring_tokens < chunk is allowed where no sequence gets longer than that.  dim_ld and vdim_ld
// are the head sizes rounded up to multiples of 8, in the projections and in the cache alike; what lies in between is zero.
//
//   prompt portions   bn_kv_gather (the chunk's tokens before the portion, out of the cache), bn_kv_prep (the portion's own,
//                     to the rows behind them and into the cache), bn_attn_chunked
//   one new token     bn_gqa_step: all of it in one launch.  A stream of the cache through warp-level MMAs, M = 16 = the
//                     query heads of a key head; a warp has its own tiles of 32 keys (TMA, 128-byte swizzle, ring of
//                     stages, softmax of its own), so no barrier runs between the first tile and the last.  CTA = (row, key
//                     head, part of the chunk); the CTA that ends last for its row and head (a ticket, nobody waits)
//                     merges the parts, and the one whose part holds the new token normalises its key, mixes its value,
//                     appends both and puts them over the stale row of its tile.
// Waits are bounded: on expiry the CTA's part is NaN, which surfaces as NaN logits, and the error word is raised.
#include "attn_portion.cuh"
#include "common.cuh"
#include "hybrid.cuh"
#include "ptx.cuh"
#include "tma.cuh"

namespace bn {

using namespace ptx;

// ---------------------------------------------------------------------------------------------------------------
// A portion's keys and values to the rows that attention reads and into the cache; a warp per (token, key head)
// ---------------------------------------------------------------------------------------------------------------
struct KvPrepParams {
    const void *k, *v, *v_first;          // columns of a projection row: [kv_heads][dim_ld], [kv_heads][vdim_ld]
    int64_t ld, v_first_ld;
    const int32_t *seq_ids, *positions;
    void *k_out, *v_out;                  // rows of kv_heads * dim_ld / vdim_ld, or null
    void *ring_k, *ring_v;
    int B, S, G, dim_ld, vdim_ld, rms_dim, rows_per_seq, row_offset, ring_tokens, chunk;
    float lambda, eps;
};

constexpr int KP_THREADS = 256;

// 8 values, one 16-byte piece in bf16 and two in fp32
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    load4(p, *reinterpret_cast<float(*)[4]>(v));
    load4(p + 4, *reinterpret_cast<float(*)[4]>(v + 4));
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
    f[0] = bf16_lo(u.x); f[1] = bf16_hi(u.x); f[2] = bf16_lo(u.y); f[3] = bf16_hi(u.y);
    f[4] = bf16_lo(u.z); f[5] = bf16_hi(u.z); f[6] = bf16_lo(u.w); f[7] = bf16_hi(u.w);
}
__device__ __forceinline__ uint4 pack8(const float (&f)[8]) {
    return make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), v); }
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) { *reinterpret_cast<uint4*>(p) = pack8(v); }

// LANES lanes (a power of two) for each (token, key head); a lane's first pieces of key, value and first value are requested
// together, heads wider than 8 LANES go round
template <typename T, int LANES>
__global__ void __launch_bounds__(KP_THREADS)
kv_prep_kernel(const KvPrepParams p) {
    grid_dependency_wait();
    grid_launch_dependents();
    constexpr int PER_BLOCK = KP_THREADS / LANES;
    const int lane = threadIdx.x % LANES;
    const unsigned n = (unsigned)p.B * p.S * p.G;
    for (unsigned at = blockIdx.x * PER_BLOCK; at < n; at += gridDim.x * PER_BLOCK) {
        const unsigned item = at + threadIdx.x / LANES;
        const bool here = item < n;                       // the whole warp takes part in the sums
        const int g = here ? (int)(item % p.G) : 0, r = here ? (int)(item / p.G) : 0;
        const int b = r / p.S, s = r - b * p.S;
        const T* k = static_cast<const T*>(p.k) + r * p.ld + g * p.dim_ld;
        const T* v = static_cast<const T*>(p.v) + r * p.ld + g * p.vdim_ld;
        const T* vf = p.v_first ? static_cast<const T*>(p.v_first) + r * p.v_first_ld + g * p.vdim_ld : nullptr;
        float k8[8] = {}, v8[8] = {}, f8[8] = {};
        const int c0 = lane * 8;
        if (here && c0 < p.dim_ld) load8(k + c0, k8);
        if (here && c0 < p.vdim_ld) {
            load8(v + c0, v8);
            if (vf) load8(vf + c0, f8);
        }
        const int start = p.positions[b], pos = start + s, last = start + p.S - 1, slot = p.seq_ids ? p.seq_ids[b] : b;
        const int64_t out_row = (int64_t)b * p.rows_per_seq + p.row_offset + s;
        T* ko = p.k_out ? static_cast<T*>(p.k_out) + (out_row * p.G + g) * p.dim_ld : nullptr;
        T* vo = p.v_out ? static_cast<T*>(p.v_out) + (out_row * p.G + g) * p.vdim_ld : nullptr;
        // only the chunk that the portion ends in is kept, so no cache row is written twice
        const int row = pos % p.chunk, first_kept = last - last % p.chunk;
        const bool keep = row < p.ring_tokens && pos >= first_kept;
        const int64_t ring_row = ((int64_t)slot * p.G + g) * p.ring_tokens + row;
        T* kr = keep ? static_cast<T*>(p.ring_k) + ring_row * p.dim_ld : nullptr;
        T* vr = keep ? static_cast<T*>(p.ring_v) + ring_row * p.vdim_ld : nullptr;
        float inv = 1.f;
        if (p.rms_dim) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(k8[e], k8[e], ss);
            for (int c = c0 + 8 * LANES; here && c < p.dim_ld; c += 8 * LANES) {
                float x[8];
                load8(k + c, x);
#pragma unroll
                for (int e = 0; e < 8; ++e) ss = fmaf(x[e], x[e], ss);
            }
#pragma unroll
            for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            inv = rsqrtf(ss / (float)p.rms_dim + p.eps);
        }
        if (!here) continue;
        for (int c = c0; c < p.dim_ld; c += 8 * LANES) {
            if (c > c0) load8(k + c, k8);
#pragma unroll
            for (int e = 0; e < 8; ++e) k8[e] *= inv;
            if (ko) store8(ko + c, k8);
            if (kr) store8(kr + c, k8);
        }
        for (int c = c0; c < p.vdim_ld; c += 8 * LANES) {
            if (c > c0) {
                load8(v + c, v8);
                if (vf) load8(vf + c, f8);
            }
            if (vf) {
#pragma unroll
                for (int e = 0; e < 8; ++e) v8[e] = fmaf(p.lambda, f8[e], (1.f - p.lambda) * v8[e]);
            }
            if (vo) store8(vo + c, v8);
            if (vr) store8(vr + c, v8);
        }
    }
}

template <typename T>
static void kv_prep_launch(const KvPrepParams& p, cudaStream_t st) {
    const int widest = p.dim_ld > p.vdim_ld ? p.dim_ld : p.vdim_ld;
    const int lanes = widest <= 64 ? 8 : widest <= 128 ? 16 : 32;
    const long long per = KP_THREADS / lanes, blocks = ((long long)p.B * p.S * p.G + per - 1) / per, cap = (long long)sm_count() * 16;
    const unsigned grid = (unsigned)(blocks < cap ? blocks : cap);
    if (lanes == 8) launch_dependent(kv_prep_kernel<T, 8>, grid, KP_THREADS, 0, st, p);
    else if (lanes == 16) launch_dependent(kv_prep_kernel<T, 16>, grid, KP_THREADS, 0, st, p);
    else launch_dependent(kv_prep_kernel<T, 32>, grid, KP_THREADS, 0, st, p);
}

// the n_old tokens of the chunk before positions[b], out of the cache, to rows 0 .. n_old - 1 of each sequence's block of
// rows; a thread moves GA_BATCH 16-byte pieces, all requested before the first is stored.  Block (pieces, key head, sequence)
constexpr int GA_THREADS = 256, GA_BATCH = 4;

__global__ void __launch_bounds__(GA_THREADS)
kv_gather_kernel(const uint4* ring_k, const uint4* ring_v, int ring_tokens, int G, int k16, int v16, const int32_t* seq_ids,
                 const int32_t* positions, int chunk, int n_old, uint4* k_out, uint4* v_out, int rows_per_seq, int blocks) {
    grid_dependency_wait();
    grid_launch_dependents();
    const int part = blockIdx.x % blocks, g = blockIdx.x / blocks % G, b = blockIdx.x / (blocks * G);
    const int slot = seq_ids ? seq_ids[b] : b, n = min(min(n_old, positions[b] % chunk), ring_tokens);    // the host sized n_old by the same positions
    const uint4* ks = ring_k + ((int64_t)slot * G + g) * ring_tokens * k16;
    const uint4* vs = ring_v + ((int64_t)slot * G + g) * ring_tokens * v16;
    uint4* kd = k_out + ((int64_t)b * rows_per_seq * G + g) * k16;
    uint4* vd = v_out + ((int64_t)b * rows_per_seq * G + g) * v16;
    const long long nk = (long long)n * k16, all = nk + (long long)n * v16;
    uint4 u[GA_BATCH];
    const long long i0 = (long long)part * GA_THREADS * GA_BATCH + threadIdx.x;
#pragma unroll
    for (int x = 0; x < GA_BATCH; ++x) {
        const long long i = i0 + x * GA_THREADS;
        if (i < all) u[x] = i < nk ? ks[i] : vs[i - nk];
    }
#pragma unroll
    for (int x = 0; x < GA_BATCH; ++x) {
        const long long i = i0 + x * GA_THREADS;
        if (i >= all) break;
        const unsigned j = (unsigned)(i < nk ? i : i - nk), w = i < nk ? k16 : v16, row = j / w;
        (i < nk ? kd : vd)[(int64_t)row * G * w + (j - row * w)] = u[x];
    }
}

// ---------------------------------------------------------------------------------------------------------------
// One new token per row
// ---------------------------------------------------------------------------------------------------------------
constexpr int ST_KEYS = 32, ST_BLK = ST_KEYS * 128;       // a 64-column block of a warp's tile: 4 KB
constexpr int ST_MAXSTAGE = 4, ST_MAXWARPS = 4, ST_MAXSPLITS = 64;
constexpr int ST_MAXDIM = 256;
constexpr int ST_SMEM_ONE = 220 * 1024, ST_SMEM_TWO = 107 * 1024;      // dynamic, for one or two CTAs per SM beside 5 KB static
constexpr float ST_LOG2E = 1.4426950408889634f;

struct StLayout {
    int nbk, nbv, warps, stages, ctas;                    // ctas: resident per SM
    int tile, q, knew, vnew, gate, ring, total;           // byte sizes and offsets
};

static StLayout st_layout(int dim_ld, int vdim_ld) {
    StLayout L;
    L.nbk = (dim_ld + 63) / 64;
    L.nbv = (vdim_ld + 63) / 64;
    L.tile = (L.nbk + L.nbv) * ST_BLK;
    L.q = 0;                                              // [16][nbk * 64 + 8] bf16
    L.knew = L.q + 16 * (L.nbk * 64 + 8) * 2;             // [nbk * 64] bf16
    L.vnew = L.knew + L.nbk * 128;                        // [nbv * 64] bf16
    L.gate = L.vnew + L.nbv * 128;                        // [16][vdim_ld] bf16
    L.ring = (L.gate + 32 * vdim_ld + 1023) / 1024 * 1024;
    const int fixed = 1024 + L.ring;
    L.warps = ST_MAXWARPS;
    for (;; L.warps /= 2) {
        const int stage = L.warps * L.tile;
        const int two = (ST_SMEM_TWO - fixed) / stage, one = (ST_SMEM_ONE - fixed) / stage;
        L.ctas = two >= 3 ? 2 : 1;
        L.stages = two >= 3 ? two : one;
        if (L.stages >= 2 || L.warps == 1) break;
    }
    if (L.stages > ST_MAXSTAGE) L.stages = ST_MAXSTAGE;
    L.total = fixed + L.warps * L.stages * L.tile;
    return L;
}

struct GqaStepParams {
    const __nv_bfloat16 *q, *k, *v, *gate, *v_first;
    int64_t ld, v_first_ld, out_ld;
    const int32_t *seq_ids, *positions;
    __nv_bfloat16 *ring_k, *ring_v, *out;
    float *part_o, *part_ml;              // [item][split][16][vdim_ld], [item][split][16][2], item = (row, key head, head group)
    int *tickets, *error_word;
    int G, rep, groups, dim_ld, vdim_ld, rms_dim, ring_tokens, chunk, splits;
    float lambda, eps, scale_log2;
    StLayout L;
};

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// NVP: 8-column pieces of the values a warp accumulates, vdim_ld <= 8 NVP.  KS: dim_ld is 16 KS and vdim_ld is 8 NVP exactly;
// 0: any sizes
template <int NVP, int KS>
__global__ void __launch_bounds__(ST_MAXWARPS * 32, 2)
gqa_step_kernel(const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_v, const GqaStepParams p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t bar[ST_MAXWARPS][ST_MAXSTAGE];
    __shared__ float s_scale[16], s_ml[ST_MAXWARPS][16][2], s_w[16][ST_MAXSPLITS];
    __shared__ int s_abort, s_last;
    const int tid = threadIdx.x, warp = tid / 32, lane = tid % 32, nw = blockDim.x / 32;
    const StLayout& L = p.L;
    const int nbk = KS ? (KS + 3) / 4 : L.nbk, nbv = KS ? (NVP + 7) / 8 : L.nbv, tile = (nbk + nbv) * ST_BLK;
    const int dim_ld = KS ? KS * 16 : p.dim_ld, vdim_ld = KS ? NVP * 8 : p.vdim_ld;
    uint8_t* base = smem_raw + (((smem_u32(smem_raw) + 1023u) & ~1023u) - smem_u32(smem_raw));
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(base + L.q);
    __nv_bfloat16* sknew = reinterpret_cast<__nv_bfloat16*>(base + L.knew);
    __nv_bfloat16* svnew = reinterpret_cast<__nv_bfloat16*>(base + L.vnew);
    __nv_bfloat16* sgate = reinterpret_cast<__nv_bfloat16*>(base + L.gate);
    const int q_ld = nbk * 64 + 8;
    uint8_t* ring = base + L.ring + warp * L.stages * tile;     // this warp's stages
    const uint32_t ring_u = smem_u32(ring);
    const int split = blockIdx.x % p.splits, item = blockIdx.x / p.splits;
    const int grp = item % p.groups, g = item / p.groups % p.G, b = item / (p.groups * p.G);
    const int h0 = g * p.rep + grp * 16, nh = min(16, p.rep - grp * 16);

    if (tid == 0) {
        for (int w = 0; w < nw; ++w)
            for (int s = 0; s < L.stages; ++s) mbar_init(smem_u32(&bar[w][s]), 1);
        s_abort = 0;
        fence_mbar_init();
        prefetch_tensormap(&tmap_k);
        prefetch_tensormap(&tmap_v);
    }
    __syncthreads();
    grid_dependency_wait();
    grid_launch_dependents();
    const int pos = p.positions[b], slot = p.seq_ids ? p.seq_ids[b] : b;
    // This warp's part of the projection row is requested before the cache is streamed, or it would arrive behind the stream.
    // A lane has 8 columns of a head.  Queries as they are (zeros beyond the group's heads and their columns), their norms go
    // into the score scale; key and value of the new token where this part may hold it
    const int c8 = lane * 8;
    const uint4 z = make_uint4(0, 0, 0, 0);
    const __nv_bfloat16* qrow = p.q + b * p.ld + h0 * dim_ld + c8;
    const __nv_bfloat16* grow = p.gate + b * p.ld + h0 * vdim_ld + c8;
    uint4 uk = z, uv = z, uf = z, uq[4], ug[4];
    auto load_heads = [&](int r0) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            uq[i] = r0 + i < nh && c8 < dim_ld ? *reinterpret_cast<const uint4*>(qrow + (r0 + i) * dim_ld) : z;
            ug[i] = p.gate && r0 + i < nh && c8 < vdim_ld ? *reinterpret_cast<const uint4*>(grow + (r0 + i) * vdim_ld) : z;
        }
    };
    load_heads(warp * 4);
    if (warp == 0 && c8 < dim_ld) uk = *reinterpret_cast<const uint4*>(p.k + b * p.ld + g * dim_ld + c8);
    if (warp == nw - 1 && c8 < vdim_ld) {
        uv = *reinterpret_cast<const uint4*>(p.v + b * p.ld + g * vdim_ld + c8);
        if (p.v_first) uf = *reinterpret_cast<const uint4*>(p.v_first + b * p.v_first_ld + g * vdim_ld + c8);
    }

    const int local = pos % p.chunk;
    const int n = local < p.ring_tokens ? local + 1 : 0;                  // keys; none: the cache has no room, the result is NaN
    const int tiles = (n + ST_KEYS - 1) / ST_KEYS, rounds = (tiles + nw - 1) / nw;
    const int per = (rounds + p.splits - 1) / p.splits * nw;
    const int t_begin = min(tiles, split * per), t_end = min(tiles, t_begin + per);
    const int row0 = (slot * p.G + g) * p.ring_tokens;
    const bool owner = t_begin < tiles && t_end == tiles;                 // this part holds the new token
    const bool new_k = owner && warp == 0, new_v = owner && warp == nw - 1;

    auto issue = [&](int t, int stage) {
        const uint32_t full = smem_u32(&bar[warp][stage]), dst = ring_u + stage * tile;
        mbar_arrive_expect_tx(full, (uint32_t)tile);
        for (int x = 0; x < nbk; ++x) tma_load_2d(dst + x * ST_BLK, &tmap_k, x * 64, row0 + t * ST_KEYS, full);
        for (int x = 0; x < nbv; ++x) tma_load_2d(dst + (nbk + x) * ST_BLK, &tmap_v, x * 64, row0 + t * ST_KEYS, full);
    };
    if (lane == 0)
        for (int s = 0; s < L.stages; ++s)
            if (t_begin + warp + s * nw < t_end) issue(t_begin + warp + s * nw, s);

    for (int r0 = warp * 4; r0 < 16; r0 += nw * 4) {
        if (r0 > warp * 4) load_heads(r0);
        float ss[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            float f[8];
            unpack8(uq[i], f);
            ss[i] = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss[i] = fmaf(f[e], f[e], ss[i]);
            if (c8 < q_ld) *reinterpret_cast<uint4*>(sq + (r0 + i) * q_ld + c8) = uq[i];
            if (c8 < vdim_ld) *reinterpret_cast<uint4*>(sgate + (r0 + i) * vdim_ld + c8) = ug[i];
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int i = 0; i < 4; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
        if (lane < 4) {
            const float t = lane == 0 ? ss[0] : lane == 1 ? ss[1] : lane == 2 ? ss[2] : ss[3];
            s_scale[r0 + lane] = p.rms_dim ? p.scale_log2 * rsqrtf(t / (float)p.rms_dim + p.eps) : p.scale_log2;
        }
    }
    if (new_k) {
        if (p.rms_dim) {
            float f[8], t = 0.f;
            unpack8(uk, f);
#pragma unroll
            for (int e = 0; e < 8; ++e) t = fmaf(f[e], f[e], t);
            const float inv = rsqrtf(warp_sum(t) / (float)p.rms_dim + p.eps);
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] *= inv;
            uk = pack8(f);
        }
        if (c8 < nbk * 64) *reinterpret_cast<uint4*>(sknew + c8) = uk;
        if (grp == 0 && c8 < dim_ld) *reinterpret_cast<uint4*>(p.ring_k + (int64_t)(row0 + local) * dim_ld + c8) = uk;
    }
    if (new_v) {
        if (p.v_first) {
            float f[8], a[8];
            unpack8(uv, f);
            unpack8(uf, a);
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = fmaf(p.lambda, a[e], (1.f - p.lambda) * f[e]);
            uv = pack8(f);
        }
        if (c8 < nbv * 64) *reinterpret_cast<uint4*>(svnew + c8) = uv;
        if (grp == 0 && c8 < vdim_ld) *reinterpret_cast<uint4*>(p.ring_v + (int64_t)(row0 + local) * vdim_ld + c8) = uv;
    }
    __syncthreads();

    const int gq = lane / 4, j = lane % 4;
    const float sc_lo = s_scale[gq], sc_hi = s_scale[gq + 8];
    const int k_steps = KS ? KS : (dim_ld + 15) / 16, npc = KS ? NVP : vdim_ld / 8;
    const uint32_t qa = smem_u32(sq) + ((lane % 16) * q_ld + (lane / 16) * 8) * 2;
    float acc[NVP][4];
#pragma unroll
    for (int i = 0; i < NVP; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    for (int t = t_begin + warp, it = 0; t < t_end; t += nw, ++it) {
        const int stage = it % L.stages;
        const uint32_t tk = ring_u + stage * tile, tv = tk + nbk * ST_BLK;
        if (__any_sync(0xffffffffu, !mbar_wait(smem_u32(&bar[warp][stage]), (it / L.stages) & 1u, &s_abort))) {
            for (int k = 1; k < L.stages && t + k * nw < t_end; ++k)        // what else is in flight, as far as it arrives
                mbar_wait(smem_u32(&bar[warp][(it + k) % L.stages]), ((it + k) / L.stages) & 1u, &s_abort);
            break;
        }
        if (t == tiles - 1) {                             // the new token's row, whatever the cache still held there
            const int r = local % ST_KEYS;
            uint8_t* at = ring + stage * tile + r * 128;
            for (int c = lane; c < (nbk + nbv) * 8; c += 32) {
                const uint4 u = c < nbk * 8 ? reinterpret_cast<const uint4*>(sknew)[c] : reinterpret_cast<const uint4*>(svnew)[c - nbk * 8];
                *reinterpret_cast<uint4*>(at + (c / 8) * ST_BLK + (((c % 8) ^ (r & 7)) << 4)) = u;
            }
            __syncwarp();
        }
        // scores: 16 heads x 32 keys
        float c[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
        const int row = (lane / 16) * 8 + lane % 8, kpart = (lane / 8) % 2;          // B fragments: keys (0-7 | 8-15) x columns (0-7 | 8-15)
        auto score_step = [&](int ks) {
            uint32_t a0, a1, a2, a3;
            ldmatrix_x4(qa + ks * 32, a0, a1, a2, a3);
            const int chunk = ks * 2 + kpart;
            const uint32_t at = tk + (chunk / 8) * ST_BLK + row * 128 + (((chunk % 8) ^ (row & 7)) << 4);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(at + half * 16 * 128, b0, b1, b2, b3);
                mma_bf16_16816(c[2 * half], a0, a1, a2, a3, b0, b1);
                mma_bf16_16816(c[2 * half + 1], a0, a1, a2, a3, b2, b3);
            }
        };
        if (KS) {
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) score_step(ks);
        } else {
#pragma unroll 4
            for (int ks = 0; ks < k_steps; ++ks) score_step(ks);
        }
        float x_lo = -INFINITY, x_hi = -INFINITY;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const bool seen = t * ST_KEYS + i * 8 + 2 * j + e < n;
                c[i][e] = seen ? c[i][e] * sc_lo : -INFINITY;
                c[i][2 + e] = seen ? c[i][2 + e] * sc_hi : -INFINITY;
                x_lo = fmaxf(x_lo, c[i][e]);
                x_hi = fmaxf(x_hi, c[i][2 + e]);
            }
#pragma unroll
        for (int o = 1; o <= 2; o *= 2) {
            x_lo = fmaxf(x_lo, __shfl_xor_sync(0xffffffffu, x_lo, o));
            x_hi = fmaxf(x_hi, __shfl_xor_sync(0xffffffffu, x_hi, o));
        }
        x_lo = fmaxf(m_lo, x_lo);                         // a tile has a key that is seen, so these are finite
        x_hi = fmaxf(m_hi, x_hi);
        const float al = ex2(m_lo - x_lo), ah = ex2(m_hi - x_hi);
        m_lo = x_lo;
        m_hi = x_hi;
        float s_lo = 0.f, s_hi = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                c[i][e] = ex2(c[i][e] - m_lo);
                c[i][2 + e] = ex2(c[i][2 + e] - m_hi);
                s_lo += c[i][e];
                s_hi += c[i][2 + e];
            }
        l_lo = fmaf(l_lo, al, s_lo);
        l_hi = fmaf(l_hi, ah, s_hi);
        if (__any_sync(0xffffffffu, al != 1.f || ah != 1.f)) {
#pragma unroll
            for (int i = 0; i < NVP; ++i) { acc[i][0] *= al; acc[i][1] *= al; acc[i][2] *= ah; acc[i][3] *= ah; }
        }
        // weighted values: the score fragments are the A operand
        uint32_t a[2][4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            a[half][0] = pack_bf16(c[2 * half][0], c[2 * half][1]);
            a[half][1] = pack_bf16(c[2 * half][2], c[2 * half][3]);
            a[half][2] = pack_bf16(c[2 * half + 1][0], c[2 * half + 1][1]);
            a[half][3] = pack_bf16(c[2 * half + 1][2], c[2 * half + 1][3]);
        }
#pragma unroll
        for (int i = 0; i < NVP; ++i) {
            if (!KS && i >= npc) break;
            uint32_t b0, b1, b2, b3;                      // 32 keys: four 8 x 8 matrices, transposed
            ldmatrix_x4_trans(tv + (i / 8) * ST_BLK + lane * 128 + (((i % 8) ^ (lane & 7)) << 4), b0, b1, b2, b3);
            mma_bf16_16816(acc[i], a[0][0], a[0][1], a[0][2], a[0][3], b0, b1);
            mma_bf16_16816(acc[i], a[1][0], a[1][1], a[1][2], a[1][3], b2, b3);
        }
        __syncwarp();
        if (lane == 0 && t + L.stages * nw < t_end) issue(t + L.stages * nw, stage);
    }
#pragma unroll
    for (int o = 1; o <= 2; o *= 2) {
        l_lo += __shfl_xor_sync(0xffffffffu, l_lo, o);
        l_hi += __shfl_xor_sync(0xffffffffu, l_hi, o);
    }
    // ---- the CTA's part: the warps' sums through shared memory (a warp's own stages; everything it asked for has arrived)
    __syncwarp();
    const int o_ld = vdim_ld + 8;
    if (s_abort == 0) {
        float* so = reinterpret_cast<float*>(ring);
#pragma unroll
        for (int i = 0; i < NVP; ++i) {
            if (!KS && i >= npc) break;
            *reinterpret_cast<float2*>(so + gq * o_ld + i * 8 + 2 * j) = make_float2(acc[i][0], acc[i][1]);
            *reinterpret_cast<float2*>(so + (gq + 8) * o_ld + i * 8 + 2 * j) = make_float2(acc[i][2], acc[i][3]);
        }
    }
    if (j == 0) {
        s_ml[warp][gq][0] = m_lo; s_ml[warp][gq][1] = l_lo;
        s_ml[warp][gq + 8][0] = m_hi; s_ml[warp][gq + 8][1] = l_hi;
    }
    __syncthreads();
    const bool bad = s_abort != 0;
    const float nan = __int_as_float(0x7fc00000);
    if (bad && tid == 0 && p.error_word) atomicExch(p.error_word, BN_ERR_TIMEOUT);
    const int quads = vdim_ld / 4;
    auto emit = [&](int r, int c4, float4 o) {            // four output columns of head r
        float f[4] = {o.x, o.y, o.z, o.w};
        if (p.gate) {
            float gt[4];
            load4(sgate + r * vdim_ld + c4, gt);
#pragma unroll
            for (int e = 0; e < 4; ++e) f[e] *= sigmoid_fast(gt[e]);
        }
        store4(p.out + b * p.out_ld + (h0 + r) * vdim_ld + c4, f);
    };
    for (int i = tid; i < nh * quads; i += blockDim.x) {
        const int r = i / quads, c4 = (i - r * quads) * 4;
        float M = -INFINITY, l = 0.f;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int w = 0; w < nw; ++w) M = fmaxf(M, s_ml[w][r][0]);
        for (int w = 0; w < nw && !bad; ++w) {
            const float f = M == -INFINITY ? 0.f : ex2(s_ml[w][r][0] - M);
            const float4 u = *reinterpret_cast<const float4*>(base + L.ring + w * L.stages * tile + (r * o_ld + c4) * 4);
            l = fmaf(s_ml[w][r][1], f, l);
            o.x = fmaf(u.x, f, o.x); o.y = fmaf(u.y, f, o.y); o.z = fmaf(u.z, f, o.z); o.w = fmaf(u.w, f, o.w);
        }
        if (p.splits == 1) {
            const float inv = bad || !(l > 0.f) ? nan : 1.f / l;
            emit(r, c4, make_float4(o.x * inv, o.y * inv, o.z * inv, o.w * inv));
        } else {
            const int64_t part = ((int64_t)item * p.splits + split) * 16 + r;
            *reinterpret_cast<float4*>(p.part_o + part * vdim_ld + c4) = o;
            if (c4 == 0) *reinterpret_cast<float2*>(p.part_ml + part * 2) = make_float2(M, bad ? nan : l);
        }
    }
    if (p.splits == 1) return;
    // ---- the last CTA of the item merges its parts
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        s_last = atomicAdd(p.tickets + item, 1) == p.splits - 1;
        if (s_last) p.tickets[item] = 0;                  // for the next launch
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    for (int r = warp; r < nh; r += nw) {
        float m2[2], l2[2], M = -INFINITY, sum = 0.f;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int s = lane + 32 * e;
            const float2 ml = s < p.splits ? __ldcg(reinterpret_cast<const float2*>(p.part_ml + (((int64_t)item * p.splits + s) * 16 + r) * 2))
                                           : make_float2(-INFINITY, 0.f);
            m2[e] = ml.x;
            l2[e] = ml.y;
            M = fmaxf(M, ml.x);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            m2[e] = m2[e] == -INFINITY ? 0.f : ex2(m2[e] - M);
            sum = fmaf(l2[e], m2[e], sum);
        }
        sum = warp_sum(sum);
        // no key at all, or a part that gave up (its sum is NaN even where its weight would be zero)
        const bool lost = !(sum > 0.f) || __any_sync(0xffffffffu, l2[0] != l2[0] || l2[1] != l2[1]);
#pragma unroll
        for (int e = 0; e < 2; ++e)
            if (lane + 32 * e < p.splits) s_w[r][lane + 32 * e] = lost ? nan : m2[e] / sum;
    }
    __syncthreads();
    for (int i = tid; i < nh * quads; i += blockDim.x) {
        const int r = i / quads, c4 = (i - r * quads) * 4;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        const float4* src = reinterpret_cast<const float4*>(p.part_o + ((int64_t)item * p.splits * 16 + r) * vdim_ld + c4);
#pragma unroll 8
        for (int s = 0; s < p.splits; ++s) {
            const float4 u = __ldcg(src + (int64_t)s * 4 * vdim_ld);
            const float f = s_w[r][s];
            o.x = fmaf(u.x, f, o.x); o.y = fmaf(u.y, f, o.y); o.z = fmaf(u.z, f, o.z); o.w = fmaf(u.w, f, o.w);
        }
        emit(r, c4, o);
    }
}

static bool gqa_step_mma_ok(int dim_ld, int vdim_ld, int dtype) {
    return dtype == 1 && dim_ld <= ST_MAXDIM && vdim_ld <= ST_MAXDIM && st_layout(dim_ld, vdim_ld).stages >= 2;
}

static bool sizes_ok(int H, int G, int dim_ld, int vdim_ld) {
    return H > 0 && G > 0 && H % G == 0 && dim_ld > 0 && vdim_ld > 0 && dim_ld % 8 == 0 && vdim_ld % 8 == 0;
}

template <int NVP, int KS>
static int gqa_step_launch(const CUtensorMap& mk, const CUtensorMap& mv, const GqaStepParams& p, unsigned grid, cudaStream_t st,
                           const char* what) {
    int dev = 0;
    cudaGetDevice(&dev);
    static thread_local int configured_dev = -1;
    if (configured_dev != dev) {
        cudaError_t e = cudaFuncSetAttribute(gqa_step_kernel<NVP, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, ST_SMEM_ONE);
        if (e != cudaSuccess) return fail(BN_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
        configured_dev = dev;
    }
    launch_dependent(gqa_step_kernel<NVP, KS>, grid, p.L.warps * 32, p.L.total, st, mk, mv, p);
    return launch_status(what);
}

}  // namespace bn

using namespace bn;

extern "C" int bn_kv_prep(const void* k, const void* v, int64_t ld, const void* v_first, int64_t v_first_ld, float lambda,
                          const int32_t* seq_ids, const int32_t* positions, int B, int S, int kv_heads, int dim_ld, int vdim_ld,
                          int rms_dim, float eps, void* k_out, void* v_out, int rows_per_seq, int row_offset, void* ring_k,
                          void* ring_v, int ring_tokens, int chunk, int dtype, bn_stream_t stream) {
    const char* what = "bn_kv_prep";
    if (!k || !v || !positions || !ring_k || !ring_v || (!k_out) != (!v_out)) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || S < 0 || !sizes_ok(kv_heads, kv_heads, dim_ld, vdim_ld) || rms_dim < 0 || rms_dim > dim_ld || ring_tokens <= 0 || chunk <= 0 ||
        (k_out && row_offset + S > rows_per_seq) || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d S=%d kv_heads=%d dim_ld=%d vdim_ld=%d chunk=%d", what, B, S, kv_heads, dim_ld,
                    vdim_ld, chunk);
    const uintptr_t all = reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(v_first) |
                          reinterpret_cast<uintptr_t>(k_out) | reinterpret_cast<uintptr_t>(v_out) | reinterpret_cast<uintptr_t>(ring_k) |
                          reinterpret_cast<uintptr_t>(ring_v);
    if ((all & 15) || ld % 8 || v_first_ld % 8) return fail(BN_ERR_INVALID_ARG, "%s: rows must start on 16-byte boundaries", what);
    if (int rc = require_sm100()) return rc;
    if (B == 0 || S == 0) return BN_OK;
    KvPrepParams p{k, v, v_first, ld, v_first_ld, seq_ids, positions, k_out, v_out, ring_k, ring_v, B, S, kv_heads, dim_ld, vdim_ld,
                   rms_dim, rows_per_seq, row_offset, ring_tokens, chunk, lambda, eps};
    if ((long long)B * S * kv_heads >= (1LL << 31)) return fail(BN_ERR_UNSUPPORTED, "%s: too many rows", what);
    if (dtype == 0) kv_prep_launch<float>(p, as_stream(stream));
    else kv_prep_launch<__nv_bfloat16>(p, as_stream(stream));
    return launch_status(what);
}

extern "C" int bn_kv_gather(const void* ring_k, const void* ring_v, int ring_tokens, int chunk, int kv_heads, int dim_ld, int vdim_ld,
                            const int32_t* seq_ids, const int32_t* positions, int B, int n_old, void* k_out, void* v_out,
                            int rows_per_seq, int dtype, bn_stream_t stream) {
    const char* what = "bn_kv_gather";
    if (!ring_k || !ring_v || !positions || !k_out || !v_out) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || n_old < 0 || n_old > ring_tokens || n_old >= chunk || n_old > rows_per_seq || !sizes_ok(kv_heads, kv_heads, dim_ld, vdim_ld) ||
        (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d n_old=%d ring_tokens=%d chunk=%d", what, B, n_old, ring_tokens, chunk);
    if ((reinterpret_cast<uintptr_t>(ring_k) | reinterpret_cast<uintptr_t>(ring_v) | reinterpret_cast<uintptr_t>(k_out) |
         reinterpret_cast<uintptr_t>(v_out)) & 15)
        return fail(BN_ERR_INVALID_ARG, "%s: pointers must be 16-byte aligned", what);
    if (int rc = require_sm100()) return rc;
    if (B == 0 || n_old == 0) return BN_OK;
    const int per = dtype == 0 ? 4 : 8, k16 = dim_ld / per, v16 = vdim_ld / per;          // 16-byte pieces of a row
    const long long pieces = (long long)n_old * (k16 + v16), blocks = (pieces + GA_THREADS * GA_BATCH - 1) / (GA_THREADS * GA_BATCH);
    if (pieces >= (1LL << 31) || blocks * B * kv_heads >= (1LL << 31)) return fail(BN_ERR_UNSUPPORTED, "%s: too many rows", what);
    launch_dependent(kv_gather_kernel, (unsigned)(blocks * B * kv_heads), GA_THREADS, 0, as_stream(stream), static_cast<const uint4*>(ring_k),
                     static_cast<const uint4*>(ring_v), ring_tokens, kv_heads, k16, v16, seq_ids, positions, chunk, n_old,
                     static_cast<uint4*>(k_out), static_cast<uint4*>(v_out), rows_per_seq, (int)blocks);
    return launch_status(what);
}

// A CTA costs its rounds of tiles plus about seven for its start and end, merging parts about five: the cut whose waves take
// the least time
extern "C" int bn_gqa_step_splits(int B, int H, int kv_heads, int dim_ld, int vdim_ld, int ring_tokens, int dtype) {
    if (B <= 0 || !sizes_ok(H, kv_heads, dim_ld, vdim_ld) || ring_tokens <= 0) return 0;
    if (!gqa_step_mma_ok(dim_ld, vdim_ld, dtype)) return 1;
    const StLayout L = st_layout(dim_ld, vdim_ld);
    const long long items = (long long)B * kv_heads * ((H / kv_heads + 15) / 16), slots = (long long)sm_count() * L.ctas;
    const int rounds = (ring_tokens + ST_KEYS * L.warps - 1) / (ST_KEYS * L.warps);
    int best = 1;
    double best_cost = 1e30;
    for (int s = 1; s <= rounds && s <= ST_MAXSPLITS; ++s) {
        const long long waves = (items * s + slots - 1) / slots;
        const double cost = (double)waves * ((rounds + s - 1) / s + 7.0) + (s > 1 ? 5.0 : 0.0) + 0.05 * s;
        if (cost < best_cost) { best_cost = cost; best = s; }
    }
    return best;
}

extern "C" int bn_gqa_step(const void* q, const void* k, const void* v, const void* gate, int64_t ld, const void* v_first,
                           int64_t v_first_ld, float lambda, void* ring_k, void* ring_v, int num_slots, int ring_tokens, int chunk,
                           const int32_t* seq_ids, const int32_t* positions, float* partial, int* tickets, int splits, void* out,
                           int64_t out_ld, int B, int H, int kv_heads, int dim_ld, int vdim_ld, int rms_dim, float eps, float scale,
                           int* error_word, int dtype, bn_stream_t stream) {
    const char* what = "bn_gqa_step";
    if (!q || !k || !v || !ring_k || !ring_v || !positions || !out) return fail(BN_ERR_INVALID_ARG, "%s: null pointer", what);
    if (B < 0 || !sizes_ok(H, kv_heads, dim_ld, vdim_ld) || rms_dim < 0 || rms_dim > dim_ld || num_slots <= 0 || ring_tokens <= 0 ||
        chunk <= 0 || splits < 1 || splits > ST_MAXSPLITS || (splits > 1 && (!partial || !tickets)) || out_ld < (int64_t)H * vdim_ld || (dtype & ~1))
        return fail(BN_ERR_INVALID_ARG, "%s: bad shape B=%d H=%d kv_heads=%d dim_ld=%d vdim_ld=%d chunk=%d ring_tokens=%d splits=%d", what, B, H,
                    kv_heads, dim_ld, vdim_ld, chunk, ring_tokens, splits);
    if ((long long)num_slots * kv_heads * ring_tokens >= (1LL << 31)) return fail(BN_ERR_UNSUPPORTED, "%s: cache of too many rows", what);
    const uintptr_t all = reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) |
                          reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(v_first) | reinterpret_cast<uintptr_t>(ring_k) |
                          reinterpret_cast<uintptr_t>(ring_v) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(partial);
    if ((all & 15) || ld % 8 || v_first_ld % 8 || out_ld % 8) return fail(BN_ERR_INVALID_ARG, "%s: rows must start on 16-byte boundaries", what);
    if (int rc = require_sm100()) return rc;
    if (B == 0) return BN_OK;
    cudaStream_t st = as_stream(stream);
    const int rep = H / kv_heads;
    if (!gqa_step_mma_ok(dim_ld, vdim_ld, dtype)) {
        // append, then one-token rows over the cache
        if (int rc = bn_kv_prep(k, v, ld, v_first, v_first_ld, lambda, seq_ids, positions, B, 1, kv_heads, dim_ld, vdim_ld, rms_dim, eps,
                                nullptr, nullptr, 0, 0, ring_k, ring_v, ring_tokens, chunk, dtype, stream))
            return rc;
        AttnPortionParams p{};
        p.q = q; p.k = ring_k; p.v = ring_v; p.gate = gate; p.out = out;
        p.q_ld = ld; p.k_ld = dim_ld; p.v_ld = vdim_ld; p.gate_ld = ld; p.out_ld = out_ld;
        p.k_head = (int64_t)ring_tokens * dim_ld; p.v_head = (int64_t)ring_tokens * vdim_ld;
        p.k_seq = kv_heads * p.k_head; p.v_seq = kv_heads * p.v_head;
        p.seq_ids = seq_ids; p.positions = positions;
        p.B = B; p.S = 1; p.rows_per_seq = ring_tokens; p.H = H; p.kv_heads = kv_heads; p.dim = dim_ld; p.vdim = vdim_ld;
        p.mask = MASK_CHUNK; p.span = chunk; p.rms_dim = rms_dim; p.rms_eps = eps; p.scale = scale;
        return attn_any(p, dtype, st, what);
    }
    CUtensorMap mk, mv;
    const uint32_t box[2] = {64, ST_KEYS};
    {
        const uint64_t dims[2] = {(uint64_t)dim_ld, (uint64_t)num_slots * kv_heads * ring_tokens}, strides[1] = {(uint64_t)dim_ld * 2};
        if (int rc = make_tensor_map(&mk, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, ring_k, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B)) return rc;
    }
    {
        const uint64_t dims[2] = {(uint64_t)vdim_ld, (uint64_t)num_slots * kv_heads * ring_tokens}, strides[1] = {(uint64_t)vdim_ld * 2};
        if (int rc = make_tensor_map(&mv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, ring_v, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B)) return rc;
    }
    GqaStepParams p{};
    p.q = static_cast<const __nv_bfloat16*>(q);
    p.k = static_cast<const __nv_bfloat16*>(k);
    p.v = static_cast<const __nv_bfloat16*>(v);
    p.gate = static_cast<const __nv_bfloat16*>(gate);
    p.v_first = static_cast<const __nv_bfloat16*>(v_first);
    p.ld = ld; p.v_first_ld = v_first_ld; p.out_ld = out_ld;
    p.seq_ids = seq_ids; p.positions = positions;
    p.ring_k = static_cast<__nv_bfloat16*>(ring_k);
    p.ring_v = static_cast<__nv_bfloat16*>(ring_v);
    p.out = static_cast<__nv_bfloat16*>(out);
    p.G = kv_heads; p.rep = rep; p.groups = (rep + 15) / 16; p.dim_ld = dim_ld; p.vdim_ld = vdim_ld; p.rms_dim = rms_dim;
    p.ring_tokens = ring_tokens; p.chunk = chunk; p.splits = splits;
    p.lambda = lambda; p.eps = eps; p.scale_log2 = scale * ST_LOG2E;
    p.tickets = tickets; p.error_word = error_word;
    const int64_t items = (int64_t)B * kv_heads * p.groups;
    p.part_o = partial;                                   // items * splits * 16 rows of vdim_ld, then of 2
    p.part_ml = partial ? partial + items * splits * 16 * vdim_ld : nullptr;
    p.L = st_layout(dim_ld, vdim_ld);
    const unsigned grid = (unsigned)(items * splits);
    if (dim_ld == 64 && vdim_ld == 64) return gqa_step_launch<8, 4>(mk, mv, p, grid, st, what);
    if (dim_ld == 128 && vdim_ld == 128) return gqa_step_launch<16, 8>(mk, mv, p, grid, st, what);
    if (vdim_ld <= 64) return gqa_step_launch<8, 0>(mk, mv, p, grid, st, what);
    if (vdim_ld <= 128) return gqa_step_launch<16, 0>(mk, mv, p, grid, st, what);
    return gqa_step_launch<32, 0>(mk, mv, p, grid, st, what);
}
