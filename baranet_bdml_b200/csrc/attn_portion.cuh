// Arguments of portion attention, shared by its any-size and its tensor-core form and by the sources that launch them.
#pragma once

#include "common.cuh"

namespace bn {

// Which keys a query sees besides none after its own: the `span` keys that end at its own, or those from the last multiple
// of `span` on (the first key row is then such a multiple)
enum { MASK_WINDOW = 0, MASK_CHUNK = 1 };

__host__ __device__ __forceinline__ int mask_oldest(int mask, int span, int own) {
    return mask == MASK_CHUNK ? own - own % span : own - span + 1;
}

// Attention of B x S query rows over key rows: row n_old + s of a sequence's rows_per_seq key rows is query s's own.  Query
// head h reads key / value head h / (H / kv_heads).
struct AttnPortionParams {
    const void *q, *k, *v, *krot;     // q (B*S, H*(dim+rot)); k (rows, kv_heads*dim), v (rows, kv_heads*vdim); krot (rows, rot), shared by the heads
    const void* gate;                 // optional (B*S, H*vdim): the result is multiplied by its sigmoid
    void* out;                        // (B*S, H*vdim)
    int64_t q_ld, k_ld, v_ld, krot_ld, gate_ld, out_ld;
    int64_t k_head, v_head;           // elements between the heads of a key / value row
    int64_t k_seq, v_seq;             // elements between the key / value rows of two sequences (any-size kernel)
    const int32_t *seq_ids, *positions;  // positions set: S = 1, sequence b's keys are those of block seq_ids[b] (null: b) up to row positions[b] % span
    int B, S, n_old, rows_per_seq, H, kv_heads, dim, rot, vdim, mask, span;
    int rms_dim;                      // > 0: queries are divided by their root mean square, the mean taken over rms_dim columns
    float rms_eps, scale;
    float score_bound;                // > 0: no scaled score is larger in magnitude
    int* error_word;                  // optional; set when a bounded wait ran out
};

bool attn_portion_sm100_ok(const AttnPortionParams& p);
int attn_portion_sm100(const AttnPortionParams& p, cudaStream_t stream);
// the kernel for any sizes; also one-token rows over a cache (positions set)
int attn_any(const AttnPortionParams& p, int dtype, cudaStream_t stream, const char* what);

}  // namespace bn
