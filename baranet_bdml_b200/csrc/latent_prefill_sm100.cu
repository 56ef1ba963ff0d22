#include "common.cuh"
#include "latent.cuh"
namespace bn {
bool attn_window_sm100_ok(const AttnWindowParams&) { return false; }
int attn_window_sm100(const AttnWindowParams&, cudaStream_t) { return fail(BN_ERR_UNSUPPORTED, "not built"); }
}
