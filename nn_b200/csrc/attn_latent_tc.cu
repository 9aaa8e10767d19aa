#include "blocks.cuh"
namespace nnq {
bool latent_tc_supported(int, int, int, int) { return false; }
nnq_status launch_latent_tc(nnq_ctx *ctx, const LatentAttn &, cudaStream_t) { return fail(ctx, NNQ_ERR_UNSUPPORTED, "not built"); }
}
