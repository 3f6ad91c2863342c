// minGRU over a prompt portion: S_t = (1 - z_t) S_(t-1) + z_t candidate_t per element.  z and the candidate depend on
// token t alone, which makes a portion a linear scan.  A CTA owns 32 elements; its warps cut the portion into segments, each warp
// composes its segment into one affine map (A, B), the maps are combined in shared memory, and every warp then walks its
// segment from the state it starts in.  f32 throughout.
#include "dense.cuh"

namespace cera {

namespace {

constexpr int SCAN_WARPS = 32, SCAN_U = 8;

template <class T>
__global__ void __launch_bounds__(SCAN_WARPS * 32) mingru_scan_kernel(const float *pre, uint32_t n, uint32_t wp, const float *__restrict__ zb,
                                                                      const float *__restrict__ xb, float *state, T *out) {
    __shared__ float sa[SCAN_WARPS][32], sb[SCAN_WARPS][32];
    pdl_trigger();
    pdl_wait();
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
    const uint32_t seg = (n + SCAN_WARPS - 1) / SCAN_WARPS, t0 = min(warp * seg, n), t1 = min(t0 + seg, n);
    const float bz = zb[c], bx = xb[c];
    const size_t ld = 3 * (size_t)wp;
    // raw products of U tokens at a time: the loads go out together
    auto walk = [&](auto step) {
        for (uint32_t t = t0; t < t1; t += SCAN_U) {
            float zr[SCAN_U], ur[SCAN_U];
#pragma unroll
            for (int u = 0; u < SCAN_U; ++u) {
                const bool in = t + u < t1;
                zr[u] = in ? pre[(t + u) * ld + c] : 0.0f;
                ur[u] = in ? pre[(t + u) * ld + wp + c] : 0.0f;
            }
            step(t, zr, ur);
        }
    };
    float A = 1.0f, B = 0.0f;
    walk([&](uint32_t t, const float *zr, const float *ur) {
#pragma unroll
        for (int u = 0; u < SCAN_U; ++u)
            if (t + u < t1) {
                float z, cand;
                mingru_gates(zr[u], ur[u], bz, bx, z, cand);
                A *= 1.0f - z;
                B = (1.0f - z) * B + z * cand;
            }
    });
    sa[warp][lane] = A;
    sb[warp][lane] = B;
    const float s0 = state[c];
    __syncthreads();
    float s = s0;
    for (uint32_t w = 0; w < warp; ++w) s = sa[w][lane] * s + sb[w][lane];
    walk([&](uint32_t t, const float *zr, const float *ur) {
        float gr[SCAN_U];
#pragma unroll
        for (int u = 0; u < SCAN_U; ++u) gr[u] = t + u < t1 ? pre[(t + u) * ld + 2 * wp + c] : 0.0f;
#pragma unroll
        for (int u = 0; u < SCAN_U; ++u)
            if (t + u < t1) {
                float z, cand;
                mingru_gates(zr[u], ur[u], bz, bx, z, cand);
                s = (1.0f - z) * s + z * cand;
                out[(size_t)(t + u) * wp + c] = Elem<T>::from(s * silu_f32(gr[u]));
            }
    });
    if (t1 == n && t0 < n) state[c] = s;  // the warp that holds the last token
}

}  // namespace

int32_t launch_mingru_scan(const float *pre, size_t n, uint32_t wp, const float *z_bias, const float *x_bias, float *state, void *out, int f32,
                           cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    count_launch();
    const dim3 grid(wp / 32), block(SCAN_WARPS * 32);
    if (f32) return check_cuda(launch_k(mingru_scan_kernel<float>, grid, block, 0, st, pre, (uint32_t)n, wp, z_bias, x_bias, state, (float *)out), "mingru scan launch");
    return check_cuda(launch_k(mingru_scan_kernel<bf16>, grid, block, 0, st, pre, (uint32_t)n, wp, z_bias, x_bias, state, (bf16 *)out), "mingru scan launch");
}

}  // namespace cera
