// Device helpers of the state-space recurrence's kernels.
#pragma once

#include "conv.cuh"

namespace cera {

// After a portion, by the CTA of values [p0, p1) of head h: the convolution's last inputs of those values, and with `shared`
// and h the first head of its group those of the group's B and C.
__device__ __forceinline__ void ssm_keep(const float *pre, const SsmView &v, uint32_t h, uint32_t p0, uint32_t p1, bool shared, uint32_t n, uint32_t start_pos,
                                         uint32_t threads) {
    const SsmShape &s = v.s;
    const uint32_t per = s.heads / s.groups, g = h / per, N = s.state_p, np = p1 - p0;
    const uint32_t total = np + (shared && h % per == 0 ? 2 * N : 0);
    for (uint32_t i = threadIdx.x; i < total; i += threads) {
        const uint32_t ch = i < np ? h * s.dim_p + p0 + i : i - np < N ? s.off_b() + g * N + i - np : s.off_c() + g * N + i - np - N;
        conv_keep(v.conv, ch, pre + s.inner_p() + ch, s.in_p, 0.0f, n, start_pos);
    }
}

}  // namespace cera
