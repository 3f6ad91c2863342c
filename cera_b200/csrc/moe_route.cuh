// Routing shared by every routed feed-forward: scores of one token's experts, the choice of the largest, and the work
// list over a batch grouped by expert (device side; launchers in moe_route.cu).
// Reference: cera/src/model/lfm2.rs:177-226 (select_experts), 673-715 (route_experts).
#pragma once

#include "common.cuh"
#include "ops.h"

namespace cera {

constexpr int MOE_MAX_EXPERTS = 256;  // the reference's stack buffer (lfm2.rs:180)
constexpr int MOE_MAX_USED = 16;

// probs[0..n_expert) hold the router logits on entry (shared memory, visible to the whole CTA) and the scores on exit.
__device__ __forceinline__ void moe_scores(float *probs, uint32_t n_expert, int softmax_gate) {
    if (softmax_gate) {
        if (threadIdx.x == 0) {
            float mx = probs[0];
            for (uint32_t e = 1; e < n_expert; ++e) mx = fmaxf(mx, probs[e]);
            float sum = 0.0f;
            for (uint32_t e = 0; e < n_expert; ++e) {
                probs[e] = expf(probs[e] - mx);
                sum += probs[e];
            }
            for (uint32_t e = 0; e < n_expert; ++e) probs[e] = probs[e] / sum;
        }
    } else {
        for (uint32_t e = threadIdx.x; e < n_expert; e += blockDim.x) probs[e] = 1.0f / (1.0f + expf(-probs[e]));
    }
    __syncthreads();
}

// One warp: the n_used experts with the largest probs + bias, ties to the lower index, in order; lane 0 writes picked /
// weight (shared memory).  Weights are the unbiased scores, divided by max(their sum, 2^-14) when `renorm`.
__device__ __forceinline__ void moe_pick(const float *probs, const float *bias, uint32_t n_expert, uint32_t n_used, int renorm, uint32_t *picked,
                                         float *weight) {
    const int lane = threadIdx.x & 31;
    uint32_t taken = 0;  // bit i: expert lane + 32 i is chosen
    float denom = 0.0f;
    for (uint32_t s = 0; s < n_used; ++s) {
        int bi = -1;
        float bv = 0.0f;
        for (uint32_t i = 0, e = lane; e < n_expert; e += 32, ++i) {
            if (taken >> i & 1) continue;
            const float v = probs[e] + (bias ? bias[e] : 0.0f);
            if (bi < 0 || v > bv) {
                bi = (int)e;
                bv = v;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (oi >= 0 && (bi < 0 || ov > bv || (ov == bv && oi < bi))) {
                bi = oi;
                bv = ov;
            }
        }
        bi = __shfl_sync(0xffffffffu, bi, 0);
        if ((bi & 31) == lane) taken |= 1u << (bi >> 5);
        if (lane == 0) {
            picked[s] = (uint32_t)bi;
            weight[s] = probs[bi];
            denom += probs[bi];
        }
    }
    if (lane == 0 && renorm) {
        denom = fmaxf(denom, 1.0f / 16384.0f);
        for (uint32_t s = 0; s < n_used; ++s) weight[s] = weight[s] / denom;
    }
    __syncwarp();
}

// Appends the work items of one expert's `c` entries starting at bucket offset `off`: items of `nc` columns go to
// the main list; a last item of at most `small_nc` columns (0 = no such list) goes to the list of narrow items at
// tiles[cap...], which a narrower kernel serves.
__device__ __forceinline__ void moe_emit_items(MoeTile *tiles, uint32_t cap, uint32_t &t, uint32_t &ts, uint32_t e, uint32_t off,
                                               uint32_t c, uint32_t nc, uint32_t small_nc) {
    for (uint32_t f = 0; f < c; f += nc) {
        const uint32_t n = c - f < nc ? c - f : nc;
        if (small_nc && n <= small_nc) tiles[cap + ts++] = MoeTile{e, off + f, n};
        else tiles[t++] = MoeTile{e, off + f, n};
    }
}

}  // namespace cera
