#include "common.cuh"
#include "mamba2.cuh"
namespace bn {
bool ssd_scan_ok(const SsmScanParams&) { return false; }
int ssd_scan(const SsmScanParams&, cudaStream_t) { return fail(BN_ERR_UNSUPPORTED, "not built"); }
}
