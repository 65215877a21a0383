#include "block_model.cuh"
namespace b200 {
bool latent_decode_fits(const LatentShape&, int) { return false; }
size_t latent_decode_scratch_floats(const LatentShape&, int) { return 0; }
int launch_latent_decode(const LatentShape&, const void*, const LatentView&, const int*, const int*, int, float*, int*, void*, cudaStream_t) { return -1; }
}
