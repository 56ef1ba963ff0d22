// Attention of a prompt portion on the 5th-generation tensor cores: keys of dim columns per key head, plus optionally one
// rotated part shared by all heads, values of another width, a sliding window or chunks, and keys that start before the
// portion's first query (the fast path of bn_attn_window and bn_attn_chunked, bf16).
//
// Persistent, one CTA per SM, eleven warps.  Work unit = (sequence, head, PAIR of 128-row query tiles); a unit walks the
// 64-key tiles from the first key that the pair's first row sees to the last row's own key:
//   warps 0-3 / 4-7   softmax of query tile 0 / 1: thread = TMEM lane = query row, 64 scores of a step in registers
//   warps 8 / 10      MMA issuer of query tile 0 / 1 (one elected thread each)
//   warp 9            TMA producer
// Shared memory holds blocks of 64 columns (128-byte swizzled rows): Q of both tiles, and a ring of K and V stages.  A
// query or key row is ceil(dim / 64) unrotated blocks and ceil(rot / 64) rotated ones; the tensor maps end at dim (keys)
// and at dim + rot (queries), so what a block holds beyond its part meets zeros on the other side.
// Tensor memory, per query tile 256 columns: 4 - nb_v score buffers of 64 columns (nb_v = 64-column blocks of the values, at
// most 3), the bf16 weights written over the scores they came from, then the output.
// Step (tile u, key tile j): S = Q K^T, softmax, O += P V.  An issuer walks the sequence of all key tiles of all units twice,
// Q K^T running as many key tiles ahead of P V as there are score buffers, across one unit's end too; per key tile its order
// is P V(j), Q K^T(j + nbuf).  The tensor pipe executes a thread's products in issue order, so new scores never overtake the
// read of the weights they replace.
// Softmax: where the caller knows a bound on the scores (unit-RMS queries and keys: dim * scale), weights are exponentials of
// the scores themselves, without a maximum; otherwise a running maximum that rescales O only when it has grown by 2^8, and
// then after the P V of the step before has landed.
// Optional: queries divided by their root mean square - a softmax thread sums its row's squares out of the Q tile and folds
// the reciprocal into the row's score scale - and outputs multiplied by the sigmoid of a gate on their way out.
// A key tile that a query tile does not see at all is skipped for that tile.  Masks are applied only by warps that have an
// edge (a row's own key, or the window's far end) inside the key tile.
// Every wait is bounded; on expiry the kernel raises the caller's error word, frees TMEM and returns.
#include "attn_portion.cuh"
#include "common.cuh"
#include "hybrid.cuh"
#include "ptx.cuh"
#include "tcgen05.cuh"
#include "tma.cuh"

namespace bn {

using namespace ptx;

constexpr int WA_BM = 128, WA_BN = 64;
constexpr int WA_THREADS = 352;
constexpr int WA_QBLK = WA_BM * 128, WA_KBLK = WA_BN * 128;      // bytes of a 64-column block
constexpr int WA_MAXSTAGE = 4;
constexpr uint32_t WA_TMEM_COLS = 512, WA_TILE_COLS = 256;
constexpr int WA_MAXVB = 3, WA_MAXBUF = 3;                       // value blocks of 64 columns, score buffers
constexpr int WA_SMEM_LIMIT = 226 * 1024;
constexpr float WA_LOG2E = 1.4426950408889634f;
constexpr float WA_RESCALE_THRESHOLD = 8.0f;                     // log2 units

struct WaParams {
    __nv_bfloat16* out;
    const __nv_bfloat16* gate;
    int64_t out_ld, gate_ld;
    int* error_word;
    int B, S, n_old, H, rep, dim, rot, vdim, mask, span, rms_dim;
    int nb_dim, nb_rot, nb_v, stages;        // 64-column blocks of the unrotated / rotated key parts and of the values
    int n_pairs, n_units, nbuf;              // nbuf: score buffers in use
    float scale_log2, rms_eps;
};

struct WaUnit {
    int b, h, i0;                            // first query row of the pair
    int key0, n;                             // first key of key tile 0; key tiles
    int first[2], last[2];                   // key tiles that query tile u needs (last < first: none)
};

__device__ __forceinline__ WaUnit wa_unit(const WaParams& p, int k) {
    WaUnit w;
    const int bh = k % (p.B * p.H);
    w.i0 = (p.n_pairs - 1 - k / (p.B * p.H)) * 2 * WA_BM;          // late rows see the most keys: they come first
    w.b = bh / p.H;
    w.h = bh - w.b * p.H;
    w.key0 = max(0, mask_oldest(p.mask, p.span, p.n_old + w.i0));
    w.n = 0;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int r0 = w.i0 + u * WA_BM;
        if (r0 >= p.S) { w.first[u] = 0; w.last[u] = -1; continue; }
        const int lo = max(0, mask_oldest(p.mask, p.span, p.n_old + r0)), hi = p.n_old + min(r0 + WA_BM, p.S) - 1;
        w.first[u] = (lo - w.key0) / WA_BN;
        w.last[u] = (hi - w.key0) / WA_BN;
        w.n = w.last[u] + 1;                                       // tile 1's last key is never before tile 0's
    }
    return w;
}

// units are dealt in snake order, so that the CTAs' sums of a descending sequence stay close
__device__ __forceinline__ int wa_unit_index(int round, int n_units) {
    const int G = gridDim.x, c = blockIdx.x;
    const int k = round * G + ((round & 1) ? G - 1 - c : c);
    return k < n_units ? k : -1;
}

// The key tiles of a CTA's units, one after the other
struct WaCursor {
    int round, j, n, first, last;            // first, last: of this cursor's query tile
    bool live;
    __device__ __forceinline__ void unit(const WaParams& p, int u) {
        const int k = wa_unit_index(round, p.n_units);
        live = k >= 0;
        j = 0;
        if (!live) return;
        const WaUnit w = wa_unit(p, k);
        n = w.n;
        first = u ? w.first[1] : w.first[0];
        last = u ? w.last[1] : w.last[0];
    }
    __device__ __forceinline__ void start(const WaParams& p, int u) { round = 0; unit(p, u); }
    __device__ __forceinline__ void next(const WaParams& p, int u) {
        if (++j < n) return;
        ++round;
        unit(p, u);
    }
    __device__ __forceinline__ bool active() const { return j >= first && j <= last; }
};

// NBK, NBV: 64-column blocks of keys and values, 0: any number
template <bool BOUNDED, int NBK, int NBV>
__global__ void __launch_bounds__(WA_THREADS, 1)
attn_portion_sm100_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                         const __grid_constant__ CUtensorMap tmap_r, const __grid_constant__ CUtensorMap tmap_v,
                         const WaParams p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t bar_q[2], bar_qfree[2], bar_s[2][WA_MAXBUF], bar_p[2][WA_MAXBUF], bar_o[2][WA_MAXBUF];
    __shared__ __align__(8) uint64_t bar_kfull[WA_MAXSTAGE], bar_kempty[WA_MAXSTAGE], bar_vfull[WA_MAXSTAGE], bar_vempty[WA_MAXSTAGE];
    __shared__ uint32_t s_tmem_base;
    __shared__ int s_abort;

    const int tid = threadIdx.x, warp = tid / 32, lane = tid % 32;
    const int nb = p.nb_dim + p.nb_rot;
    const uint32_t smem0 = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t sQ = smem0, sK = smem0 + 2 * nb * WA_QBLK, sV = sK + p.stages * nb * WA_KBLK;

    if (tid == 0) {
        for (int u = 0; u < 2; ++u) {
            mbar_init(smem_u32(&bar_q[u]), 1);
            mbar_init(smem_u32(&bar_qfree[u]), p.rms_dim ? 5 : 1);      // the last Q K^T, and the softmax warps that read Q
            for (int x = 0; x < WA_MAXBUF; ++x) {
                mbar_init(smem_u32(&bar_s[u][x]), 1);
                mbar_init(smem_u32(&bar_p[u][x]), 128);
                mbar_init(smem_u32(&bar_o[u][x]), 1);
            }
        }
        for (int s = 0; s < WA_MAXSTAGE; ++s) {
            mbar_init(smem_u32(&bar_kfull[s]), 1);
            mbar_init(smem_u32(&bar_kempty[s]), 2);               // both issuers
            mbar_init(smem_u32(&bar_vfull[s]), 1);
            mbar_init(smem_u32(&bar_vempty[s]), 2);
        }
        s_abort = 0;
        fence_mbar_init();
    }
    if (warp == 8) {
        tc::tmem_alloc(smem_u32(&s_tmem_base), WA_TMEM_COLS);
        tc::tmem_relinquish();
    }
    tc::fence_before_sync();
    __syncthreads();
    tc::fence_after_sync();
    const uint32_t tmem = s_tmem_base;

    if (warp == 9) {
        // ---------------------------------------------------------- TMA producer
        if (lane == 0) {
            prefetch_tensormap(&tmap_q);
            prefetch_tensormap(&tmap_k);
            prefetch_tensormap(&tmap_r);
            prefetch_tensormap(&tmap_v);
            bool ok = true;
            int stage = 0;
            uint32_t phase = 0, nq[2] = {0, 0};              // nq: query tiles loaded so far
            for (int round = 0; ok; ++round) {
                const int k = wa_unit_index(round, p.n_units);
                if (k < 0) break;
                const WaUnit w = wa_unit(p, k);
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    if (!ok || w.last[u] < w.first[u]) continue;
                    ok = mbar_wait(smem_u32(&bar_qfree[u]), (nq[u] & 1u) ^ 1u, &s_abort);
                    if (!ok) continue;
                    ++nq[u];
                    mbar_arrive_expect_tx(smem_u32(&bar_q[u]), nb * WA_QBLK);
                    for (int x = 0; x < nb; ++x) {
                        const int col = x < p.nb_dim ? x * 64 : p.dim + (x - p.nb_dim) * 64;
                        tma_load_4d(sQ + (u * nb + x) * WA_QBLK, &tmap_q, col, w.h, w.i0 + u * WA_BM, w.b, smem_u32(&bar_q[u]));
                    }
                }
                for (int j = 0; ok && j < w.n; ++j) {
                    const int key = w.key0 + j * WA_BN;
                    ok = mbar_wait(smem_u32(&bar_kempty[stage]), phase ^ 1u, &s_abort);
                    if (!ok) break;
                    mbar_arrive_expect_tx(smem_u32(&bar_kfull[stage]), nb * WA_KBLK);
                    for (int x = 0; x < p.nb_dim; ++x)
                        tma_load_4d(sK + (stage * nb + x) * WA_KBLK, &tmap_k, x * 64, w.h / p.rep, key, w.b, smem_u32(&bar_kfull[stage]));
                    for (int x = 0; x < p.nb_rot; ++x)
                        tma_load_4d(sK + (stage * nb + p.nb_dim + x) * WA_KBLK, &tmap_r, x * 64, 0, key, w.b, smem_u32(&bar_kfull[stage]));
                    ok = mbar_wait(smem_u32(&bar_vempty[stage]), phase ^ 1u, &s_abort);
                    if (!ok) break;
                    mbar_arrive_expect_tx(smem_u32(&bar_vfull[stage]), p.nb_v * WA_KBLK);
                    for (int x = 0; x < p.nb_v; ++x)
                        tma_load_4d(sV + (stage * p.nb_v + x) * WA_KBLK, &tmap_v, x * 64, w.h / p.rep, key, w.b, smem_u32(&bar_vfull[stage]));
                    if (++stage == p.stages) { stage = 0; phase ^= 1u; }
                }
            }
        }
    } else if (warp >= 8) {
        // ------------------------------------------------------------ MMA issuers
        // one thread per query tile (a thread's issue rate, not the tensor pipe, would bound one thread for both); descriptors are
        // stepped as their low words, block and step counts are compile-time for the common sizes
        constexpr uint32_t IDESC_QK = tc::idesc_bf16(WA_BM, WA_BN, 0), IDESC_PV = tc::idesc_bf16(WA_BM, 64, 1);
        constexpr uint32_t DESC_HI = (uint32_t)(tc::smem_desc_sw128(0) >> 32), DESC_LO = (uint32_t)tc::smem_desc_sw128(0);
        if (elect_one()) {
            const int u = warp == 8 ? 0 : 1;
            const int nbv = NBV ? NBV : p.nb_v;
            const uint32_t tT = tmem + u * WA_TILE_COLS, tO = tT + WA_TILE_COLS - nbv * 64;
            const uint32_t dq = DESC_LO + (sQ >> 4) + u * nb * (WA_QBLK >> 4), dK = DESC_LO + (sK >> 4), dV = DESC_LO + (sV >> 4);
            const uint32_t aS = smem_u32(bar_s[u]), aP = smem_u32(bar_p[u]), aO = smem_u32(bar_o[u]), aQ = smem_u32(&bar_q[u]),
                           aQf = smem_u32(&bar_qfree[u]), aKf = smem_u32(bar_kfull), aKe = smem_u32(bar_kempty), aVf = smem_u32(bar_vfull),
                           aVe = smem_u32(bar_vempty);
            bool ok = true;
            uint32_t kstage = 0, vstage = 0, kphase = 0, vphase = 0, qbuf = 0, pbuf = 0, pphase = 0, nq = 0;
            WaCursor cq, cp;                                         // Q K^T, P V
            cq.start(p, u);
            cp.start(p, u);
            int ahead = 0;                                           // key tiles with Q K^T issued and P V not
            while (cq.live || ahead > 0) {
                // Q K^T stays within one unit of P V: the queries of the unit after that are loaded only when the softmax warps
                // have read this unit's, which they do after they have put out the unit before
                const bool qk = cq.live && cq.round <= cp.round + 1, pv = ahead == p.nbuf || !qk;
                if (pv) {                                            // O += P V
                    // a tile also waits for key tiles that it does not see: a stage's release counts both tiles, once per filling
                    ok = mbar_wait(aVf + vstage * 8, vphase, &s_abort);
                    if (!ok) break;
                    if (cp.active()) {
                        ok = mbar_wait(aP + pbuf * 8, pphase, &s_abort);
                        if (!ok) break;
                        tc::fence_after_sync();
                        const uint32_t tP = tT + pbuf * WA_BN, more = cp.j > cp.first;
                        const uint32_t dv = dV + vstage * nbv * (WA_KBLK >> 4);
                        if (NBV) {
#pragma unroll
                            for (int x = 0; x < NBV; ++x)
#pragma unroll
                                for (int kk = 0; kk < WA_BN / 16; ++kk)
                                    tc::mma_ts_lohi(tO + x * 64, tP + kk * 8, dv + x * (WA_KBLK >> 4) + kk * 128, DESC_HI, IDESC_PV,
                                                    kk > 0 ? 1u : more);
                        } else {
                            for (int x = 0; x < nbv; ++x)
#pragma unroll
                                for (int kk = 0; kk < WA_BN / 16; ++kk)
                                    tc::mma_ts_lohi(tO + x * 64, tP + kk * 8, dv + x * (WA_KBLK >> 4) + kk * 128, DESC_HI, IDESC_PV,
                                                    kk > 0 ? 1u : more);
                        }
                        if (BOUNDED) {
                            if (cp.j == cp.last) tc::commit(aO);
                        } else {
                            tc::commit(aO + pbuf * 8);
                        }
                        if (++pbuf == p.nbuf) { pbuf = 0; pphase ^= 1u; }
                    }
                    tc::commit(aVe + vstage * 8);
                    if (++vstage == p.stages) { vstage = 0; vphase ^= 1u; }
                    cp.next(p, u);
                }
                if (qk) {                                            // S = Q K^T
                    ok = mbar_wait(aKf + kstage * 8, kphase, &s_abort);
                    if (!ok) break;
                    if (cq.active()) {
                        if (cq.j == cq.first) {
                            ok = mbar_wait(aQ, nq & 1u, &s_abort);
                            ++nq;
                            if (!ok) break;
                        }
                        tc::fence_after_sync();
                        const uint32_t tS = tT + qbuf * WA_BN, dk = dK + kstage * nb * (WA_KBLK >> 4);
                        if (NBK) {
                            // what a block holds beyond its part is zero, or meets zeros: every block takes four steps
#pragma unroll
                            for (int x = 0; x < NBK; ++x)
#pragma unroll
                                for (int kk = 0; kk < 4; ++kk)
                                    tc::mma_ss_lohi(tS, dq + x * (WA_QBLK >> 4) + kk * 2, dk + x * (WA_KBLK >> 4) + kk * 2, DESC_HI, IDESC_QK,
                                                    x > 0 || kk > 0);
                        } else {
                            uint32_t more = 0;
                            for (int x = 0; x < nb; ++x) {
                                const int cols = x < p.nb_dim ? p.dim - x * 64 : p.rot - (x - p.nb_dim) * 64;
                                const int steps = cols >= 64 ? 4 : (cols + 15) / 16;
                                for (int kk = 0; kk < steps; ++kk) {
                                    tc::mma_ss_lohi(tS, dq + x * (WA_QBLK >> 4) + kk * 2, dk + x * (WA_KBLK >> 4) + kk * 2, DESC_HI, IDESC_QK,
                                                    more);
                                    more = 1;
                                }
                            }
                        }
                        tc::commit(aS + qbuf * 8);
                        if (cq.j == cq.last) tc::commit(aQf);
                        if (++qbuf == p.nbuf) qbuf = 0;
                    }
                    tc::commit(aKe + kstage * 8);
                    if (++kstage == p.stages) { kstage = 0; kphase ^= 1u; }
                    cq.next(p, u);
                }
                ahead += (int)qk - (int)pv;
            }
        }
        __syncwarp();
    } else {
        // ---------------------------------------------------------- softmax warps
        const int u = warp / 4;
        const uint32_t lane_base = ((uint32_t)((warp % 4) * 32)) << 16;
        const uint32_t tT = tmem + lane_base + u * WA_TILE_COLS, tO = tT + WA_TILE_COLS - p.nb_v * 64;
        bool ok = true;
        int buf = 0;
        uint32_t phase = 0, nu = 0, nq = 0;                          // nu: units so far
        // the latest P V that this query tile has handed its weights to: an output barrier per score buffer where every step
        // may have to wait for one (two phases of a barrier are then never outstanding), else one per unit
        auto wait_pv = [&]() {
            if (BOUNDED) return mbar_wait(smem_u32(&bar_o[u][0]), nu & 1u, &s_abort);
            return buf == 0 ? mbar_wait(smem_u32(&bar_o[u][p.nbuf - 1]), phase ^ 1u, &s_abort)
                            : mbar_wait(smem_u32(&bar_o[u][buf - 1]), phase, &s_abort);
        };
        for (int round = 0; ok; ++round) {
            const int k = wa_unit_index(round, p.n_units);
            if (k < 0) break;
            const WaUnit w = wa_unit(p, k);
            const int first = u ? w.first[1] : w.first[0], last = u ? w.last[1] : w.last[0];
            if (last < first) continue;
            const int row0 = w.i0 + u * WA_BM + (warp % 4) * 32;     // the warp's first row
            const int gi = row0 + lane;
            const int own = p.n_old + gi, oldest = mask_oldest(p.mask, p.span, own);         // the keys this row sees
            const int warp_own0 = p.n_old + row0, warp_oldest1 = mask_oldest(p.mask, p.span, warp_own0 + 31);
            float scale_log2 = p.scale_log2;
            if (p.rms_dim) {
                ok = mbar_wait(smem_u32(&bar_q[u]), nq & 1u, &s_abort);
                ++nq;
                if (!ok) break;
                const uint8_t* qrow = smem_raw + (sQ - smem_u32(smem_raw)) + u * nb * WA_QBLK + ((warp % 4) * 32 + lane) * 128;
                float s0 = 0.f, s1 = 0.f;
                for (int x = 0; x < p.nb_dim; ++x) {
#pragma unroll
                    for (int i = 0; i < 8; ++i) {      // the row's 16-byte pieces in an order without bank conflicts
                        const uint4 v = *reinterpret_cast<const uint4*>(qrow + x * WA_QBLK + ((i ^ (lane & 7)) << 4));
                        s0 = fmaf(bf16_lo(v.x), bf16_lo(v.x), s0); s1 = fmaf(bf16_hi(v.x), bf16_hi(v.x), s1);
                        s0 = fmaf(bf16_lo(v.y), bf16_lo(v.y), s0); s1 = fmaf(bf16_hi(v.y), bf16_hi(v.y), s1);
                        s0 = fmaf(bf16_lo(v.z), bf16_lo(v.z), s0); s1 = fmaf(bf16_hi(v.z), bf16_hi(v.z), s1);
                        s0 = fmaf(bf16_lo(v.w), bf16_lo(v.w), s0); s1 = fmaf(bf16_hi(v.w), bf16_hi(v.w), s1);
                    }
                }
                scale_log2 *= rsqrtf((s0 + s1) / (float)p.rms_dim + p.rms_eps);
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(&bar_qfree[u]));
            }
            float m_ref = -INFINITY;
            float l0 = 0.f, l1 = 0.f, l2 = 0.f, l3 = 0.f;
            for (int j = first; j <= last; ++j) {
                ok = mbar_wait(smem_u32(&bar_s[u][buf]), phase, &s_abort);
                if (!ok) break;
                tc::fence_after_sync();
                const uint32_t tS = tT + buf * WA_BN;
                const int key = w.key0 + j * WA_BN;
                const bool masked = key + WA_BN - 1 > warp_own0 || key < warp_oldest1;
                uint32_t r[2][32];
                tc::ld32(tS, r[0]);
                tc::ld32(tS + 32, r[1]);
                tc::wait_ld(r[0]);
                tc::wait_ld(r[1]);
                if (masked) {
#pragma unroll
                    for (int c = 0; c < 2; ++c)
#pragma unroll
                        for (int i = 0; i < 32; ++i) {
                            const int kk = key + c * 32 + i;
                            if (kk > own || kk < oldest) r[c][i] = 0xff800000u;          // -inf
                        }
                }
                float mneg = 0.f;
                if (!BOUNDED) {
                    float t0 = -INFINITY, t1 = -INFINITY, t2 = -INFINITY, t3 = -INFINITY;
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        t0 = fmaxf(t0, __uint_as_float(r[0][i]));
                        t1 = fmaxf(t1, __uint_as_float(r[0][i + 1]));
                        t2 = fmaxf(t2, __uint_as_float(r[1][i]));
                        t3 = fmaxf(t3, __uint_as_float(r[1][i + 1]));
                    }
                    const float m_new = fmaxf(m_ref, fmaxf(fmaxf(t0, t1), fmaxf(t2, t3)));
                    const bool grow = (m_new - m_ref) * scale_log2 > WA_RESCALE_THRESHOLD;   // NaN (both -inf) is false
                    if (__any_sync(0xffffffffu, grow)) {
                        if (j > first) {
                            ok = wait_pv();                          // of the step before
                            if (!ok) break;
                            tc::fence_after_sync();
                            const float alpha = m_ref == -INFINITY ? 0.f : ex2((m_ref - m_new) * scale_log2);
                            l0 *= alpha; l1 *= alpha; l2 *= alpha; l3 *= alpha;
#pragma unroll 1
                            for (int c = 0; c < 4 * p.nb_v; ++c) {
                                uint32_t o[16];
                                tc::ld16(tO + c * 16, o);
                                tc::wait_ld(o);
#pragma unroll
                                for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                                tc::st16(tO + c * 16, o);
                            }
                        }
                        m_ref = m_new;
                    }
                    // a row that has seen no key yet has only -inf scores: any finite reference gives zero weights
                    mneg = m_ref == -INFINITY ? 0.f : -m_ref * scale_log2;
                }
                if (BOUNDED) {
                    const uint64_t sc2 = pack_f32x2(scale_log2, scale_log2), zero2 = pack_f32x2(0.f, 0.f);
                    uint64_t la = pack_f32x2(l0, l1), lb = pack_f32x2(l2, l3);
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        uint32_t pk[16];
#pragma unroll
                        for (int i = 0; i < 32; i += 2) {
                            float p0, p1;
                            unpack_f32x2(fma_f32x2(pack_f32x2(__uint_as_float(r[c][i]), __uint_as_float(r[c][i + 1])), sc2, zero2), p0, p1);
                            p0 = ex2(p0);
                            p1 = ex2(p1);
                            if (i & 2) lb = add_f32x2(lb, pack_f32x2(p0, p1));
                            else la = add_f32x2(la, pack_f32x2(p0, p1));
                            pk[i / 2] = pack_bf16(p0, p1);
                        }
                        tc::st16(tS + c * 16, pk);
                    }
                    unpack_f32x2(la, l0, l1);
                    unpack_f32x2(lb, l2, l3);
                } else {
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        uint32_t pk[16];
#pragma unroll
                        for (int i = 0; i < 32; i += 2) {
                            const float p0 = ex2(fmaf(__uint_as_float(r[c][i]), scale_log2, mneg));
                            const float p1 = ex2(fmaf(__uint_as_float(r[c][i + 1]), scale_log2, mneg));
                            l0 += p0;
                            l1 += p1;
                            pk[i / 2] = pack_bf16(p0, p1);
                        }
                        tc::st16(tS + c * 16, pk);
                    }
                }
                tc::wait_st();
                tc::fence_before_sync();
                mbar_arrive(smem_u32(&bar_p[u][buf]));
                if (++buf == p.nbuf) { buf = 0; phase ^= 1u; }
            }
            if (!ok) break;
            // O / l, gated -> bf16 -> global
            const float l_run = (l0 + l1) + (l2 + l3);
            const __nv_bfloat16* gate = p.gate && gi < p.S ? p.gate + ((int64_t)w.b * p.S + gi) * p.gate_ld + w.h * p.vdim : nullptr;
            uint4 g4[4];
            auto load_gate = [&](int c) {                            // of 32 columns, requested before they are needed
#pragma unroll
                for (int v = 0; v < 4; ++v)
                    if (gate && c * 32 + v * 8 < p.vdim) g4[v] = *reinterpret_cast<const uint4*>(gate + c * 32 + v * 8);
            };
            load_gate(0);
            ok = wait_pv();
            ++nu;
            if (!ok) break;
            tc::fence_after_sync();
            const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
            __nv_bfloat16* dst = p.out + ((int64_t)w.b * p.S + gi) * p.out_ld + w.h * p.vdim;
            for (int c = 0; c < 2 * p.nb_v; ++c) {
                uint32_t o[32];
                tc::ld32(tO + c * 32, o);
                tc::wait_ld(o);
                if (gi < p.S) {
#pragma unroll
                    for (int v = 0; v < 4; ++v)
                        if (c * 32 + v * 8 < p.vdim) {                 // vdim is a multiple of 8
                            float f[8];
#pragma unroll
                            for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(o[v * 8 + e]) * inv;
                            if (gate) {
                                const uint32_t gw[4] = {g4[v].x, g4[v].y, g4[v].z, g4[v].w};
#pragma unroll
                                for (int e = 0; e < 4; ++e) {
                                    f[2 * e] *= sigmoid_fast(bf16_lo(gw[e]));
                                    f[2 * e + 1] *= sigmoid_fast(bf16_hi(gw[e]));
                                }
                            }
                            *reinterpret_cast<uint4*>(dst + c * 32 + v * 8) =
                                make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
                        }
                    load_gate(c + 1);
                }
            }
            // the next unit's first PV overwrites O: it waits for this warp's next arrival on bar_p, which follows
            tc::fence_before_sync();
        }
    }

    // common exit: everybody arrives here (all waits are bounded), then TMEM is freed
    tc::fence_before_sync();
    __syncthreads();
    if (tid == 0 && s_abort && p.error_word) atomicExch(p.error_word, BN_ERR_TIMEOUT);
    if (warp == 8) {
        tc::fence_after_sync();
        tc::tmem_dealloc(tmem, WA_TMEM_COLS);
    }
}

static int wa_stages(int nb, int nb_v) {
    const int left = WA_SMEM_LIMIT - 1024 - 2 * nb * WA_QBLK;
    const int per = (nb + nb_v) * WA_KBLK;
    const int s = left > 0 ? left / per : 0;
    return s > WA_MAXSTAGE ? WA_MAXSTAGE : s;
}

bool attn_portion_sm100_ok(const AttnPortionParams& p) {
    const int nb = (p.dim + 63) / 64 + (p.rot + 63) / 64, nb_v = (p.vdim + 63) / 64;
    const uintptr_t bases = reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.k) | reinterpret_cast<uintptr_t>(p.v) |
                            reinterpret_cast<uintptr_t>(p.krot) | reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.out);
    const int64_t strides = p.q_ld | p.k_ld | p.v_ld | p.krot_ld | p.gate_ld | p.out_ld | p.k_head | p.v_head;
    return ((p.dim | p.rot | p.vdim | strides) & 7) == 0 && (bases & 15) == 0 && !(p.rms_dim && p.rot) && !p.positions &&
           nb_v <= WA_MAXVB && wa_stages(nb, nb_v) >= 2 && p.scale > 0.f;
}

static int wa_map(CUtensorMap* m, const void* base, int inner, int heads, int64_t head_stride, int rows, int64_t ld, int B, int box_rows) {
    const uint64_t dims[4] = {(uint64_t)inner, (uint64_t)heads, (uint64_t)rows, (uint64_t)B};
    const uint64_t strides[3] = {(uint64_t)head_stride * 2, (uint64_t)ld * 2, (uint64_t)ld * 2 * rows};
    const uint32_t box[4] = {64, 1, (uint32_t)box_rows, 1};
    return make_tensor_map(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, base, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
}

template <bool BOUNDED, int NBK, int NBV>
static int wa_launch(unsigned grid, size_t smem, cudaStream_t st, const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mr,
                     const CUtensorMap& mv, const WaParams& p, int dev, const char* what) {
    static thread_local int configured_dev = -1;
    if (configured_dev != dev) {
        cudaError_t e = cudaFuncSetAttribute(attn_portion_sm100_kernel<BOUNDED, NBK, NBV>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             WA_SMEM_LIMIT);
        if (e != cudaSuccess) return fail(BN_ERR_CUDA, "%s: %s", what, cudaGetErrorString(e));
        configured_dev = dev;
    }
    attn_portion_sm100_kernel<BOUNDED, NBK, NBV><<<grid, WA_THREADS, smem, st>>>(mq, mk, mr, mv, p);
    return launch_status(what);
}

int attn_portion_sm100(const AttnPortionParams& a, cudaStream_t st) {
    const char* what = "portion attention";
    CUtensorMap mq, mk, mr, mv;
    if (int rc = wa_map(&mq, a.q, a.dim + a.rot, a.H, a.dim + a.rot, a.S, a.q_ld, a.B, WA_BM)) return rc;
    if (int rc = wa_map(&mk, a.k, a.dim, a.kv_heads, a.k_head, a.rows_per_seq, a.k_ld, a.B, WA_BN)) return rc;
    mr = mk;                                                           // without a rotated part nothing reads it
    if (a.rot)
        if (int rc = wa_map(&mr, a.krot, a.rot, 1, a.krot_ld, a.rows_per_seq, a.krot_ld, a.B, WA_BN)) return rc;
    if (int rc = wa_map(&mv, a.v, a.vdim, a.kv_heads, a.v_head, a.rows_per_seq, a.v_ld, a.B, WA_BN)) return rc;
    WaParams p;
    p.out = static_cast<__nv_bfloat16*>(a.out);
    p.out_ld = a.out_ld;
    p.error_word = a.error_word;
    p.gate = static_cast<const __nv_bfloat16*>(a.gate);
    p.gate_ld = a.gate_ld;
    p.B = a.B; p.S = a.S; p.n_old = a.n_old; p.H = a.H; p.rep = a.H / a.kv_heads; p.dim = a.dim; p.rot = a.rot; p.vdim = a.vdim;
    p.mask = a.mask; p.span = a.span; p.rms_dim = a.rms_dim; p.rms_eps = a.rms_eps;
    p.nb_dim = (a.dim + 63) / 64;
    p.nb_rot = (a.rot + 63) / 64;
    p.nb_v = (a.vdim + 63) / 64;
    p.stages = wa_stages(p.nb_dim + p.nb_rot, p.nb_v);
    p.n_pairs = (a.S + 2 * WA_BM - 1) / (2 * WA_BM);
    const long long units = (long long)a.B * a.H * p.n_pairs;
    if (units > (1 << 30)) return fail(BN_ERR_UNSUPPORTED, "%s: too many query tiles", what);
    p.n_units = (int)units;
    p.nbuf = 4 - p.nb_v < p.stages ? 4 - p.nb_v : p.stages;
    p.scale_log2 = a.scale * WA_LOG2E;
    // the weights of a row are at most 2^60 and at least 2^-60, their sums far from either end of fp32
    const bool bounded = a.score_bound > 0.f && a.score_bound * WA_LOG2E <= 60.f;
    const int nb = p.nb_dim + p.nb_rot;
    const size_t smem = 1024 + (size_t)2 * nb * WA_QBLK + (size_t)p.stages * (nb + p.nb_v) * WA_KBLK;
    int dev = 0, sms = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const unsigned grid = (unsigned)(p.n_units < sms ? p.n_units : sms);
    const int sizes = nb * 4 + p.nb_v;
    if (bounded && sizes == 1 * 4 + 1) return wa_launch<true, 1, 1>(grid, smem, st, mq, mk, mr, mv, p, dev, what);
    if (bounded && sizes == 2 * 4 + 2) return wa_launch<true, 2, 2>(grid, smem, st, mq, mk, mr, mv, p, dev, what);
    if (bounded) return wa_launch<true, 0, 0>(grid, smem, st, mq, mk, mr, mv, p, dev, what);
    if (sizes == 1 * 4 + 1) return wa_launch<false, 1, 1>(grid, smem, st, mq, mk, mr, mv, p, dev, what);
    if (sizes == 2 * 4 + 2) return wa_launch<false, 2, 2>(grid, smem, st, mq, mk, mr, mv, p, dev, what);
    if (sizes == 3 * 4 + 2) return wa_launch<false, 3, 2>(grid, smem, st, mq, mk, mr, mv, p, dev, what);
    return wa_launch<false, 0, 0>(grid, smem, st, mq, mk, mr, mv, p, dev, what);
}

}  // namespace bn
