#include "latent_attention.cuh"
namespace plz {
bool latent_tc_fits(int, int) { return false; }
int latent_tc_rows(int rows) { return 64; }
int launch_latent_tc(const LatentAttnArgs&, const LatentParams&, cudaStream_t) { return PLZ_ERR_UNSUPPORTED; }
}
