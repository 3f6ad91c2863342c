// Element-type helpers of the dense kernels: 16-byte vectors of T and their f32 values.
#pragma once

#include "dense.h"

namespace cera {

using bf16 = __nv_bfloat16;

template <class T>
struct Elem;
template <>
struct Elem<bf16> {
    static constexpr int N = 8;  // elements of a 16-byte vector
    static __device__ __forceinline__ void unpack(const uint4 &v, float (&f)[8]) {
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
        }
    }
    static __device__ __forceinline__ float to(bf16 v) { return __bfloat162float(v); }
    static __device__ __forceinline__ bf16 from(float v) { return __float2bfloat16_rn(v); }
};
template <>
struct Elem<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void unpack(const uint4 &v, float (&f)[4]) {
        f[0] = __uint_as_float(v.x);
        f[1] = __uint_as_float(v.y);
        f[2] = __uint_as_float(v.z);
        f[3] = __uint_as_float(v.w);
    }
    static __device__ __forceinline__ float to(float v) { return v; }
    static __device__ __forceinline__ float from(float v) { return v; }
};

__device__ __forceinline__ void store4(float *p, const float4 &v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(bf16 *p, const float4 &v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}

__device__ __forceinline__ float sigmoid_f32(float x) { return __fdividef(1.0f, 1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x * sigmoid_f32(x); }
__device__ __forceinline__ float softplus_f32(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
// min(g, limit) * sigmoid(alpha g) * (clamp(u) + shift)
__device__ __forceinline__ float gated_unit(float g, float u, const ExpertAct &a) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
    return g * sigmoid_f32(a.alpha * g) * (u + a.shift);
}
// minGRU: gate z and candidate from their raw products
__device__ __forceinline__ void mingru_gates(float zr, float ur, float zb, float ub, float &z, float &cand) {
    z = sigmoid_f32(zr + zb);
    const float u = ur + ub;
    cand = u >= 0.0f ? u + 0.5f : sigmoid_f32(u);
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
// Sum over the CTA (red: 33 floats of shared memory, reusable after the call by the next one).
__device__ __forceinline__ float cta_sum(float v, float *red) {
    v = warp_sum(v);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n = blockDim.x >> 5;
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    if (warp == 0) {
        v = lane < n ? red[lane] : 0.0f;
        v = warp_sum(v);
        if (lane == 0) red[32] = v;
    }
    __syncthreads();
    return red[32];
}

}  // namespace cera
