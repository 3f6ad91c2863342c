// The short causal convolution's device side: one position, and moving the ring on.
#pragma once

#include "dense.cuh"

namespace cera {

// Channel ch at position pos from its own input and the ring.  The ring's row of pos itself is not read: whoever keeps the
// new input may write it while others still convolve.
__device__ __forceinline__ float conv_one(const ConvView &c, uint32_t ch, uint32_t pos, float now) {
    const float *w = c.w + (size_t)ch * c.taps;
    float acc = c.bias[ch];
    uint32_t slot = (pos + 1) % c.taps;
    for (uint32_t k = 0; k + 1 < c.taps; ++k) {
        acc = fmaf(w[k], c.ring[(size_t)slot * c.channels + ch], acc);
        slot = slot + 1 == c.taps ? 0 : slot + 1;
    }
    return fmaf(w[c.taps - 1], now, acc);
}

// After a portion of n positions: the last inputs of channel ch go into the ring.
__device__ __forceinline__ void conv_keep(const ConvView &c, uint32_t ch, const float *in, size_t ld_in, float in_bias, uint32_t n, uint32_t start_pos) {
    for (uint32_t t = n > c.taps ? n - c.taps : 0; t < n; ++t)
        c.ring[(size_t)((start_pos + t) % c.taps) * c.channels + ch] = in[(size_t)t * ld_in] + in_bias;
}

}  // namespace cera
