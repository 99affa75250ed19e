#include "latent.cuh"
namespace tbl { namespace stack {
bool latent_tensor_supported(const tbl_latent_mixer&) { return false; }
int latent_tensor_heads(const tbl_latent_mixer&) { return 16; }
cudaError_t launch_latent_tensor(const LatentParams&, int, cudaStream_t) { return cudaErrorNotSupported; }
} }
