// What the latent-attention sources share: launch arguments and the choice between the any-size kernels and the
// tensor-core ones.
#pragma once

#include "common.cuh"

namespace bn {

inline int round8(int v) { return (v + 7) / 8 * 8; }

// Attention of B x S query rows over expanded keys: row n_old + s of a sequence's rows_per_seq key rows is query s's own
struct AttnWindowParams {
    const void *q, *k, *v, *krot;     // q (B*S, H*(dim+rot)); k (rows, H*dim) and v (rows, H*vdim) with one row stride; krot (rows, rot)
    void* out;                        // (B*S, H*vdim)
    int64_t q_ld, kv_ld, krot_ld, out_ld;
    int B, S, n_old, rows_per_seq, H, dim, rot, vdim, window;
    float scale;
    int* error_word;                  // optional; set when a bounded wait ran out
};

struct LatentDecodeParams {
    const void *q_abs, *ring;
    const int32_t *seq_ids, *positions;
    float *partial, *lse;             // [B][H][splits][kv_ld], [B][H][splits]
    int B, H, kv_ld, rot_ld, num_slots, ring_tokens, window, splits;
    float scale;
};

bool attn_window_sm100_ok(const AttnWindowParams& p);
int attn_window_sm100(const AttnWindowParams& p, cudaStream_t stream);
bool latent_decode_mma_ok(int H, int kv_ld, int rot_ld);
int latent_decode_mma_splits(int B, int H, int window, int sms);
int latent_decode_mma(const LatentDecodeParams& p, cudaStream_t stream);
// bf16 forms of bn_latent_absorb_q and bn_latent_expand_out; false when the sizes or alignments are not theirs
bool latent_absorb_mma(const void* q, int64_t q_ld, const void* wuk, const double* freq, const int32_t* positions, void* q_abs, int B,
                       int H, int dim, int rot, int kv_ld, int rot_ld, cudaStream_t stream);
bool latent_expand_mma(float* partial, const float* lse, int splits, const void* wuv, void* out, int64_t out_ld, int B, int H,
                       int vdim, int kv_ld, cudaStream_t stream);

}  // namespace bn
