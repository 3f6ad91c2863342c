#include "dense.cuh"
namespace cera {
int32_t launch_dense_gemm_tc(const DenseGemm &, cudaStream_t, bool *taken) { *taken = false; return CERA_CUDA_OK; }
}
