#include "latent.cuh"
namespace tbl { namespace stack {
bool latent_expanded_supported(const tbl_latent_mixer&) { return false; }
int launch_latent_expanded(const tbl_latent_mixer&, const LatentParams&, int, int, cudaStream_t) { return TBL_ERR_UNSUPPORTED; }
} }
