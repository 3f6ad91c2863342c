// The short causal convolution over a prompt portion.  A thread owns one channel and a run of positions and slides the
// inputs through registers; positions before the portion come from the ring.
#include "conv.cuh"

namespace cera {

namespace {

constexpr uint32_t CV_RUN = 32;

// TAPS 0: any number (inputs are read again for every tap)
template <class T, int TAPS>
__global__ void __launch_bounds__(128) conv_kernel(const float *in, size_t ld_in, const float *__restrict__ in_bias, ConvView c, int silu, uint32_t n,
                                                   uint32_t start_pos, T *out, size_t ld_out) {
    pdl_trigger();
    const uint32_t ch = blockIdx.x * 128 + threadIdx.x, t0 = blockIdx.y * CV_RUN, t1 = min(t0 + CV_RUN, n);
    if (ch >= c.channels) return;
    const float bias = c.bias[ch], ib = in_bias ? in_bias[ch] : 0.0f;
    const int taps = TAPS ? TAPS : (int)c.taps;
    const float *w = c.w + (size_t)ch * taps;
    float wk[TAPS ? TAPS : 1], win[TAPS ? TAPS : 1];
#pragma unroll
    for (int k = 0; k < TAPS; ++k) wk[k] = w[k];
    pdl_wait();
    auto input = [&](int t) {  // of position start_pos + t
        return t >= 0 ? in[(size_t)t * ld_in + ch] + ib : c.ring[(size_t)((start_pos + taps + t) % taps) * c.channels + ch];
    };
    auto store = [&](uint32_t t, float v) { out[(size_t)t * ld_out + ch] = Elem<T>::from(silu ? silu_f32(v) : v); };
    if constexpr (TAPS != 0) {
#pragma unroll
        for (int k = 0; k + 1 < TAPS; ++k) win[k + 1] = input((int)t0 - (TAPS - 1 - k));
        for (uint32_t t = t0; t < t1; t += 8) {
            float now[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) now[u] = t + u < t1 ? input((int)(t + u)) : 0.0f;
#pragma unroll
            for (int u = 0; u < 8; ++u) {
#pragma unroll
                for (int k = 0; k + 1 < TAPS; ++k) win[k] = win[k + 1];
                win[TAPS - 1] = now[u];
                float acc = bias;
#pragma unroll
                for (int k = 0; k < TAPS; ++k) acc = fmaf(wk[k], win[k], acc);
                if (t + u < t1) store(t + u, acc);
            }
        }
    } else {
        for (uint32_t t = t0; t < t1; ++t) {
            float acc = bias;
            for (int k = 0; k < taps; ++k) acc = fmaf(w[k], input((int)t - (taps - 1 - k)), acc);
            store(t, acc);
        }
    }
}

}  // namespace

int32_t launch_conv(const float *in, size_t ld_in, const float *in_bias, const ConvView &c, int silu, size_t n, size_t start_pos, void *out, size_t ld_out,
                    int f32, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    const dim3 grid((c.channels + 127) / 128, (unsigned)((n + CV_RUN - 1) / CV_RUN));
    auto go = [&](auto kernel, auto *o) {
        count_launch();
        return check_cuda(launch_k(kernel, grid, dim3(128), 0, st, in, ld_in, in_bias, c, silu, (uint32_t)n, (uint32_t)start_pos, o, ld_out), "convolution launch");
    };
    auto typed = [&](auto *o) {
        using T = std::remove_pointer_t<decltype(o)>;
        switch (c.taps) {
            case 2: return go(conv_kernel<T, 2>, o);
            case 3: return go(conv_kernel<T, 3>, o);
            case 4: return go(conv_kernel<T, 4>, o);
            default: return go(conv_kernel<T, 0>, o);
        }
    };
    return f32 ? typed((float *)out) : typed((bf16 *)out);
}

}  // namespace cera
