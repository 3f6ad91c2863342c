#include "dense.cuh"
namespace cera {
bool latent_prefill_supports(const LatentShape &) { return false; }
int32_t launch_latent_prefill(const void *, const LatentShape &, const void *, const void *, size_t, const void *, size_t, const float *, const float *, size_t, size_t, void *, size_t, cudaStream_t, bool *taken) { *taken = false; return CERA_CUDA_OK; }
}
