// Greedy pick: the first maximum of the logits (cera/src/sampler.rs:20-30), two stages.
#include <cmath>

#include "ops.h"

namespace cera {

namespace {

constexpr int ARGMAX_BLOCKS = 128, ARGMAX_THREADS = 256;

// Order: greater value wins; on equal values the lower index wins, which is
// what a left-to-right strict `>` scan returns.
__device__ __forceinline__ void amax_merge(float &bv, uint32_t &bi, float v, uint32_t i) {
    if (v > bv || (v == bv && i < bi)) {
        bv = v;
        bi = i;
    }
}

__global__ void argmax_stage1(const float *__restrict__ x, uint32_t n, uint32_t *scratch) {
    pdl_trigger();
    pdl_wait();
    float bv = -INFINITY;
    uint32_t bi = 0xFFFFFFFFu;
    for (uint32_t i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
        const float v = x[i];
        if (v > bv) {  // ascending i within a thread: strict > keeps the first
            bv = v;
            bi = i;
        }
    }
    __shared__ float sv[ARGMAX_THREADS];
    __shared__ uint32_t si[ARGMAX_THREADS];
    sv[threadIdx.x] = bv;
    si[threadIdx.x] = bi;
    __syncthreads();
    for (int s = blockDim.x / 2; s > 0; s >>= 1) {
        if ((int)threadIdx.x < s) amax_merge(sv[threadIdx.x], si[threadIdx.x], sv[threadIdx.x + s], si[threadIdx.x + s]);
        __syncthreads();
    }
    if (threadIdx.x == 0) {
        scratch[2 * blockIdx.x] = __float_as_uint(sv[0]);
        scratch[2 * blockIdx.x + 1] = si[0];
    }
}

__global__ void argmax_stage2(const uint32_t *__restrict__ scratch, int blocks, uint32_t *out) {
    pdl_trigger();
    pdl_wait();
    float bv = -INFINITY;
    uint32_t bi = 0xFFFFFFFFu;
    for (int b = threadIdx.x; b < blocks; b += 32) amax_merge(bv, bi, __uint_as_float(scratch[2 * b]), scratch[2 * b + 1]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const uint32_t oi = __shfl_xor_sync(0xffffffffu, bi, o);
        amax_merge(bv, bi, ov, oi);
    }
    // no finite / non-NaN winner -> index 0, as the reference returns
    if (threadIdx.x == 0) *out = bi == 0xFFFFFFFFu ? 0u : bi;
}

}  // namespace

size_t argmax_scratch_words() { return 2 * ARGMAX_BLOCKS; }

int32_t launch_argmax(const float *x, size_t n, uint32_t *out, uint32_t *scratch, cudaStream_t st) {
    if (!x || !out || !scratch) return fail(CERA_CUDA_ERR_BAD_ARG, "argmax: null argument");
    count_launch(2);
    CERA_CUDA_TRY(launch_k(argmax_stage1, dim3(ARGMAX_BLOCKS), dim3(ARGMAX_THREADS), 0, st, x, (uint32_t)n, scratch));
    return check_cuda(launch_k(argmax_stage2, dim3(1), dim3(32), 0, st, (const uint32_t *)scratch, (int)ARGMAX_BLOCKS, out),
                      "argmax launch");
}

}  // namespace cera
