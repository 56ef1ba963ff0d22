// Launch arguments shared by the token-by-token scan and the chunked tensor-core scan.
#pragma once

#include "common.cuh"

namespace bn {

struct SsmScanParams {
    const void* xbc;                  // (rows, xbc_ld): [x: H*P | B: G*N | C: G*N], convolved
    const float *dt, *a, *D;          // (rows, H) step sizes and log decays; (H)
    float* state;                     // [slot][H][P][N]
    const int32_t* seq_ids;
    void* y;                          // (rows, y_ld)
    int64_t xbc_ld, y_ld;
    int B, S, H, P, G, N;
};

bool ssd_scan_ok(const SsmScanParams& p);
int ssd_scan(const SsmScanParams& p, cudaStream_t stream);

}  // namespace bn
