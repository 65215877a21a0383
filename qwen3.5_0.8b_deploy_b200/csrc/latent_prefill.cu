#include "block_model.cuh"
namespace b200 {
bool latent_prefill_fits(const LatentShape&) { return false; }
int launch_latent_prefill(const LatentShape&, const void*, int, const void*, const void*, const void*, int, const LatentTile*, int, void*, int*, cudaStream_t) { return -1; }
}
