// Real-gated linear recurrent unit (Griffin): S = a S + sqrt(1 - a^2) i u per channel, where u is a convolved projection,
// log a = -decay * r * softplus(lam), and the gates r, i are block-diagonal products of u through a sigmoid.  The output is
// S * gelu(y) with a second projection y.
//
// Decode: one kernel takes the raw products of both branches; a CTA convolves its block's channels, a warp forms both gates
// of a channel and moves its state on.  Portion: convolution (conv.cu) and gates (a block-diagonal product) come first; a and
// the input term depend on one token alone, so the portion is a linear scan cut into segments as in mingru.cu.  States,
// decays and gates are f32.
#include "conv.cuh"
#include "dense_gemv.cuh"

namespace cera {

namespace {

using namespace gv;

__device__ __forceinline__ float gelu_tanh_f32(float x) {
    // 0.5 (1 + tanh z) = sigmoid(2 z)
    return x * sigmoid_f32(2.0f * 0.79788456080286535588f * (x + 0.044715f * x * x * x));
}
// log a, a - 1 and the input term's factor from the raw gates; sp = decay * softplus(lam).  Slow channels have a within a few
// units of rounding of 1: a - 1 keeps what a itself would lose, step after step.
__device__ __forceinline__ void rglru_gates(float r_raw, float i_raw, float sp, float &log_a, float &am1, float &gain) {
    log_a = -sp * sigmoid_f32(r_raw);
    am1 = expm1f(log_a);
    gain = sqrtf(-am1 * (2.0f + am1)) * sigmoid_f32(i_raw);  // 1 - a^2 = (1 - a)(1 + a)
}
// a s + input
__device__ __forceinline__ float decayed(float am1, float s, float input) { return s + fmaf(am1, s, input); }

// grid (groups of 8 channels of a block, blocks)
template <class T>
__global__ void __launch_bounds__(GV_WARPS * 32) rglru_step_kernel(const float *pre, RglruView v, const uint32_t *pos_dev, T *out) {
    extern __shared__ __align__(16) uint8_t smem[];
    T *us = reinterpret_cast<T *>(smem);  // the block's convolved channels
    pdl_trigger();
    const uint32_t b = blockIdx.y, bp = v.block_p, lane = threadIdx.x & 31, c = blockIdx.x * GV_WARPS + (threadIdx.x >> 5);  // channel of the block
    RowDot<T, 2, 2> d;
    d.w[0] = (const T *)v.gates.w + ((size_t)b * 2 * bp + c) * bp;
    d.w[1] = d.w[0] + (size_t)bp * bp;
    d.start(bp, 0, 1);
    d.fetch();
    const uint32_t ch = b * bp + c;
    const float sp = v.decay * softplus_f32(v.lam[ch]);
    pdl_wait();
    const uint32_t pos = *pos_dev;
    for (uint32_t i = threadIdx.x; i < bp; i += GV_WARPS * 32) {
        const uint32_t k = b * bp + i;
        const float now = pre[v.wp + k] + v.in_bias[v.wp + k];
        us[i] = Elem<T>::from(conv_one(v.conv, k, pos, now));
        if (blockIdx.x == 0) v.conv.ring[(size_t)(pos % v.conv.taps) * v.conv.channels + k] = now;
    }
    __syncthreads();
    float acc[2] = {};
    d.run(us, acc);
    group_sum<2, 1>(acc, nullptr);
    if (lane == 0) {
        float log_a, am1, gain;
        rglru_gates(acc[0] + v.gate_bias[(size_t)b * 2 * bp + c], acc[1] + v.gate_bias[(size_t)b * 2 * bp + bp + c], sp, log_a, am1, gain);
        const float s = decayed(am1, v.state[ch], gain * Elem<T>::to(us[c]));
        v.state[ch] = s;
        out[ch] = Elem<T>::from(s * gelu_tanh_f32(pre[ch] + v.in_bias[ch]));
    }
}

constexpr int RG_WARPS = 32, RG_U = 8;

template <class T>
__global__ void __launch_bounds__(RG_WARPS * 32) rglru_scan_kernel(const float *pre, const T *u, const float *gate, RglruView v, uint32_t n, uint32_t start_pos,
                                                                   T *out) {
    __shared__ float sa[RG_WARPS][32], sb[RG_WARPS][32];
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane, wp = v.wp, bp = v.block_p;
    const uint32_t seg = (n + RG_WARPS - 1) / RG_WARPS, t0 = min(warp * seg, n), t1 = min(t0 + seg, n);
    const uint32_t gr = c / bp * 2 * bp + c % bp, gi = gr + bp;  // this channel among the gates' rows
    const float br = v.gate_bias[gr], bi = v.gate_bias[gi], by = v.in_bias[c], sp = v.decay * softplus_f32(v.lam[c]);
    const size_t ld = 2 * (size_t)wp;
    pdl_wait();
    auto walk = [&](auto step) {  // RG_U tokens at a time: the loads go out together
        for (uint32_t t = t0; t < t1; t += RG_U) {
            float r[RG_U], i[RG_U], x[RG_U];
#pragma unroll
            for (int k = 0; k < RG_U; ++k) {
                const bool in = t + k < t1;
                r[k] = in ? gate[(t + k) * ld + gr] : 0.0f;
                i[k] = in ? gate[(t + k) * ld + gi] : 0.0f;
                x[k] = in ? Elem<T>::to(u[(size_t)(t + k) * wp + c]) : 0.0f;
            }
            step(t, r, i, x);
        }
    };
    float A = 0.0f, B = 0.0f;  // a segment: s -> e^A s + B
    walk([&](uint32_t t, const float *r, const float *i, const float *x) {
#pragma unroll
        for (int k = 0; k < RG_U; ++k)
            if (t + k < t1) {
                float log_a, am1, gain;
                rglru_gates(r[k] + br, i[k] + bi, sp, log_a, am1, gain);
                A += log_a;
                B = decayed(am1, B, gain * x[k]);
            }
    });
    sa[warp][lane] = expm1f(A);
    sb[warp][lane] = B;
    const float s0 = v.state[c];
    __syncthreads();
    float s = s0;
    for (uint32_t w = 0; w < warp; ++w) s = decayed(sa[w][lane], s, sb[w][lane]);
    walk([&](uint32_t t, const float *r, const float *i, const float *x) {
        float y[RG_U];
#pragma unroll
        for (int k = 0; k < RG_U; ++k) y[k] = t + k < t1 ? pre[(t + k) * ld + c] : 0.0f;
#pragma unroll
        for (int k = 0; k < RG_U; ++k)
            if (t + k < t1) {
                float log_a, am1, gain;
                rglru_gates(r[k] + br, i[k] + bi, sp, log_a, am1, gain);
                s = decayed(am1, s, gain * x[k]);
                out[(size_t)(t + k) * wp + c] = Elem<T>::from(s * gelu_tanh_f32(y[k] + by));
            }
    });
    if (t1 == n && t0 < n) v.state[c] = s;  // the warp that holds the last token
    if (warp == 0) conv_keep(v.conv, c, pre + wp + c, ld, v.in_bias[wp + c], n, start_pos);
}

}  // namespace

int32_t launch_rglru_step(const float *pre, const RglruView &v, const uint32_t *pos_dev, void *out, cudaStream_t st) {
    const dim3 grid(v.block_p / GV_WARPS, v.wp / v.block_p);
    count_launch();
    return with_type(v.gates.f32, [&](auto t) {
        using T = decltype(t);
        return check_cuda(launch_k(rglru_step_kernel<T>, grid, dim3(GV_WARPS * 32), v.block_p * sizeof(T), st, pre, v, pos_dev, (T *)out), "rglru step launch");
    });
}

int32_t launch_rglru_scan(const float *pre, const void *u, const float *gate, const RglruView &v, size_t n, size_t start_pos, void *out, int f32,
                          cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    count_launch();
    return with_type(f32, [&](auto t) {
        using T = decltype(t);
        return check_cuda(launch_k(rglru_scan_kernel<T>, dim3(v.wp / 32), dim3(RG_WARPS * 32), 0, st, pre, (const T *)u, gate, v, (uint32_t)n,
                                   (uint32_t)start_pos, (T *)out),
                          "rglru scan launch");
    });
}

}  // namespace cera
