#include "block_model.cuh"
namespace b200 {
bool mlstm_chunk_fits(const MlstmShape&) { return false; }
int launch_mlstm_chunk(const MlstmShape&, const void*, int, const float*, int, const float*, const LaSeqMeta*, int, int, float*, float*, int*, cudaStream_t) { return -1; }
}
