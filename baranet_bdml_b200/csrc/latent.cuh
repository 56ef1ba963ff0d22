// What the latent-attention sources share: launch arguments and the choice between the any-size kernels and the
// tensor-core ones.
#pragma once

#include "common.cuh"

namespace bn {

inline int round8(int v) { return (v + 7) / 8 * 8; }

struct LatentDecodeParams {
    const void *q_abs, *ring;
    const int32_t *seq_ids, *positions;
    float *partial, *lse;             // [B][H][splits][kv_ld], [B][H][splits]
    int B, H, kv_ld, rot_ld, num_slots, ring_tokens, window, splits;
    float scale;
};

bool latent_decode_mma_ok(int H, int kv_ld, int rot_ld);
int latent_decode_mma_splits(int B, int H, int window, int sms);
int latent_decode_mma(const LatentDecodeParams& p, cudaStream_t stream);
// bf16 forms of bn_latent_absorb_q and bn_latent_expand_out; false when the sizes or alignments are not theirs
bool latent_absorb_mma(const void* q, int64_t q_ld, const void* wuk, const double* freq, const int32_t* positions, void* q_abs, int B,
                       int H, int dim, int rot, int kv_ld, int rot_ld, cudaStream_t stream);
bool latent_expand_mma(float* partial, const float* lse, int splits, const void* wuv, void* out, int64_t out_ld, int B, int H,
                       int vdim, int kv_ld, cudaStream_t stream);

}  // namespace bn
