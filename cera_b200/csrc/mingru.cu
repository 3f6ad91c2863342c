// minGRU over a prompt portion: S_t = (1 - z_t) S_(t-1) + z_t candidate_t per element, gates read from the current token
// only, so a portion is a linear scan.  A CTA owns 32 elements; its warps cut the portion into segments, each warp
// composes its segment into one affine map (A, B), the maps are combined in shared memory, and every warp then walks its
// segment from the state it starts in.  f32 throughout.
#include "dense.cuh"

namespace cera {

namespace {

constexpr int SCAN_WARPS = 32;

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
    float A = 1.0f, B = 0.0f;
    for (uint32_t t = t0; t < t1; ++t) {
        float z, cand;
        mingru_gates(pre[t * ld + c], pre[t * ld + wp + c], bz, bx, z, cand);
        A *= 1.0f - z;
        B = (1.0f - z) * B + z * cand;
    }
    sa[warp][lane] = A;
    sb[warp][lane] = B;
    const float s0 = state[c];
    __syncthreads();
    float s = s0;
    for (uint32_t w = 0; w < warp; ++w) s = sa[w][lane] * s + sb[w][lane];
    for (uint32_t t = t0; t < t1; ++t) {
        float z, cand;
        mingru_gates(pre[t * ld + c], pre[t * ld + wp + c], bz, bx, z, cand);
        s = (1.0f - z) * s + z * cand;
        out[(size_t)t * wp + c] = Elem<T>::from(s * silu_f32(pre[t * ld + 2 * wp + c]));
    }
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
