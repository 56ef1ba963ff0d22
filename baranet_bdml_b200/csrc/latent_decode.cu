#include "common.cuh"
#include "latent.cuh"
namespace bn {
bool latent_decode_mma_ok(int, int, int) { return false; }
int latent_decode_mma_splits(int, int, int, int) { return 1; }
int latent_decode_mma(const LatentDecodeParams&, cudaStream_t) { return fail(BN_ERR_UNSUPPORTED, "not built"); }
}
