// Routing launchers shared by the routed feed-forwards (moe.cu, layered.cu): scores and picks of a batch, and the work
// list that groups its (token, pick) pairs by expert.
#include "moe_route.cuh"

namespace cera {

namespace {

// One CTA per token.  Warps take experts round-robin; lane-strided f32 dot, shuffle tree.
__global__ void __launch_bounds__(256) moe_route_kernel(const float *x, const float *__restrict__ router,
                                                        const float *__restrict__ bias, uint32_t hidden, uint32_t ld_x, uint32_t n_expert,
                                                        uint32_t n_used, int softmax_gate, int renorm, uint32_t *ids, float *weights,
                                                        uint32_t *counts) {
    __shared__ float probs[MOE_MAX_EXPERTS];
    __shared__ uint32_t picked[MOE_MAX_USED];
    __shared__ float w[MOE_MAX_USED];
    pdl_trigger();
    pdl_wait();
    const uint32_t j = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float *xj = x + (size_t)j * ld_x;
    for (uint32_t e = warp; e < n_expert; e += blockDim.x >> 5) {
        const float *r = router + (size_t)e * hidden;
        float acc = 0.0f;
        for (uint32_t i = lane; i < hidden; i += 32) acc = fmaf(r[i], xj[i], acc);
        acc = warp_sum(acc);
        if (lane == 0) probs[e] = acc;
    }
    __syncthreads();
    moe_scores(probs, n_expert, softmax_gate);
    if (warp != 0) return;
    moe_pick(probs, bias, n_expert, n_used, renorm, picked, w);
    if (lane < n_used) {
        ids[(size_t)j * n_used + lane] = picked[lane];
        weights[(size_t)j * n_used + lane] = w[lane];
        atomicAdd(counts + picked[lane], 1u);
    }
}

// One CTA: bucket offsets, cursors, and the work lists (n_tiles[0] main, n_tiles[1] narrow).  counts is zeroed again
// for the next call.
__global__ void moe_plan_kernel(uint32_t *counts, uint32_t n_expert, uint32_t nc, uint32_t small_nc, uint32_t cap, uint32_t *cursor,
                                MoeTile *tiles, uint32_t *n_tiles) {
    pdl_trigger();
    pdl_wait();
    if (threadIdx.x != 0) return;
    uint32_t off = 0, t = 0, ts = 0;
    for (uint32_t e = 0; e < n_expert; ++e) {
        const uint32_t c = counts[e];
        cursor[e] = off;
        moe_emit_items(tiles, cap, t, ts, e, off, c, nc, small_nc);
        off += c;
        counts[e] = 0;
    }
    n_tiles[0] = t;
    n_tiles[1] = ts;
}

}  // namespace

int32_t launch_moe_route(const float *x, size_t ld_x, size_t n, const float *router, const float *bias, uint32_t hidden, uint32_t n_expert,
                         uint32_t n_used, int softmax_gate, int renorm, uint32_t *ids, float *weights, uint32_t *counts, cudaStream_t st) {
    if (n_expert == 0 || n_expert > MOE_MAX_EXPERTS || n_used == 0 || n_used > MOE_MAX_USED || n_used > n_expert)
        return fail(CERA_CUDA_ERR_BAD_ARG, "moe route: %u experts, %u used (limits %d, %d)", n_expert, n_used, MOE_MAX_EXPERTS, MOE_MAX_USED);
    if (n == 0) return CERA_CUDA_OK;
    count_launch();
    return check_cuda(launch_k(moe_route_kernel, dim3((unsigned)n), dim3(256), 0, st, x, router, bias, hidden, (uint32_t)ld_x, n_expert, n_used,
                               softmax_gate, renorm, ids, weights, counts),
                      "moe route launch");
}

int32_t launch_moe_plan(uint32_t *counts, uint32_t n_expert, uint32_t nc, uint32_t small_nc, uint32_t cap, uint32_t *cursor, MoeTile *tiles,
                        uint32_t *n_tiles, cudaStream_t st) {
    count_launch();
    return check_cuda(launch_k(moe_plan_kernel, dim3(1), dim3(32), 0, st, counts, n_expert, nc, small_nc, cap, cursor, tiles, n_tiles), "moe plan launch");
}

}  // namespace cera
