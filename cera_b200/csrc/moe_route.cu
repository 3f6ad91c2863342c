// Routing launchers shared by the routed feed-forwards (moe.cu, layered.cu): scores and picks of a batch, and the work
// list that groups its (token, pick) pairs by expert.
#include "moe_route.cuh"

namespace cera {

namespace {

// One CTA per T tokens.  A warp takes four experts at a time: lane-strided float4 dots in f32, every router and token
// vector loaded once for the 4 T products it enters; shuffle tree; then warp t picks for token t.
template <int T>
__global__ void __launch_bounds__(256) moe_route_kernel(const float *x, const float *__restrict__ router,
                                                        const float *__restrict__ bias, uint32_t hidden, uint32_t ld_x, uint32_t n, uint32_t n_expert,
                                                        uint32_t n_used, int softmax_gate, int renorm, uint32_t *ids, float *weights,
                                                        uint32_t *counts) {
    __shared__ float probs[T][MOE_MAX_EXPERTS];
    __shared__ uint32_t picked[T][MOE_MAX_USED];
    __shared__ float w[T][MOE_MAX_USED];
    pdl_trigger();
    pdl_wait();
    const uint32_t j0 = blockIdx.x * T;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float *xj[T];
#pragma unroll
    for (int t = 0; t < T; ++t) xj[t] = x + (size_t)min(j0 + t, n - 1) * ld_x;
    constexpr int EG = 4;
    for (uint32_t e0 = warp * EG; e0 < n_expert; e0 += (blockDim.x >> 5) * EG) {
        const float4 *r[EG];
#pragma unroll
        for (int g = 0; g < EG; ++g) r[g] = reinterpret_cast<const float4 *>(router + (size_t)min(e0 + g, n_expert - 1) * hidden);
        float acc[EG][T] = {};
        for (uint32_t i = lane; i < hidden / 4; i += 32) {
            float4 rv[EG];
#pragma unroll
            for (int g = 0; g < EG; ++g) rv[g] = __ldg(r[g] + i);
#pragma unroll
            for (int t = 0; t < T; ++t) {
                const float4 xv = reinterpret_cast<const float4 *>(xj[t])[i];
#pragma unroll
                for (int g = 0; g < EG; ++g)
                    acc[g][t] = fmaf(rv[g].w, xv.w, fmaf(rv[g].z, xv.z, fmaf(rv[g].y, xv.y, fmaf(rv[g].x, xv.x, acc[g][t]))));
            }
        }
#pragma unroll
        for (int g = 0; g < EG; ++g)
#pragma unroll
            for (int t = 0; t < T; ++t) {
                const float v = warp_sum(acc[g][t]);
                if (lane == 0 && e0 + g < n_expert) probs[t][e0 + g] = v;
            }
    }
    __syncthreads();
#pragma unroll 1
    for (int t = 0; t < T; ++t) moe_scores(probs[t], n_expert, softmax_gate);
    if (warp >= T || j0 + warp >= n) return;
    const uint32_t j = j0 + warp;
    moe_pick(probs[warp], bias, n_expert, n_used, renorm, picked[warp], w[warp]);
    if (lane < n_used) {
        ids[(size_t)j * n_used + lane] = picked[warp][lane];
        weights[(size_t)j * n_used + lane] = w[warp][lane];
        atomicAdd(counts + picked[warp][lane], 1u);
    }
}

// One CTA: bucket offsets, cursors, and the work lists (n_tiles[0] main, n_tiles[1] narrow).  counts is zeroed again
// for the next call.
__global__ void moe_plan_kernel(uint32_t *counts, uint32_t n_expert, uint32_t nc, uint32_t small_nc, uint32_t cap, uint32_t *cursor,
                                MoeTile *tiles, uint32_t *n_tiles) {
    pdl_trigger();
    pdl_wait();
    __shared__ uint32_t n_of[MOE_MAX_EXPERTS];
    for (uint32_t e = threadIdx.x; e < n_expert; e += blockDim.x) {
        n_of[e] = counts[e];
        counts[e] = 0;
    }
    __syncthreads();
    if (threadIdx.x != 0) return;
    uint32_t off = 0, t = 0, ts = 0;
    for (uint32_t e = 0; e < n_expert; ++e) {
        const uint32_t c = n_of[e];
        cursor[e] = off;
        moe_emit_items(tiles, cap, t, ts, e, off, c, nc, small_nc);
        off += c;
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
    auto go = [&](auto kernel, uint32_t per) {
        return check_cuda(launch_k(kernel, dim3((unsigned)((n + per - 1) / per)), dim3(256), 0, st, x, router, bias, hidden, (uint32_t)ld_x, (uint32_t)n, n_expert,
                                   n_used, softmax_gate, renorm, ids, weights, counts),
                          "moe route launch");
    };
    return n < (size_t)sm_count() * 4 ? go(moe_route_kernel<1>, 1) : go(moe_route_kernel<8>, 8);
}

int32_t launch_moe_plan(uint32_t *counts, uint32_t n_expert, uint32_t nc, uint32_t small_nc, uint32_t cap, uint32_t *cursor, MoeTile *tiles,
                        uint32_t *n_tiles, cudaStream_t st) {
    count_launch();
    return check_cuda(launch_k(moe_plan_kernel, dim3(1), dim3(32), 0, st, counts, n_expert, nc, small_nc, cap, cursor, tiles, n_tiles), "moe plan launch");
}

}  // namespace cera
