// State-space recurrence with a matrix state per head (Mamba-2): S = exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x,
// dt = softplus(raw + bias); x, B, C come convolved through silu, B and C are shared by the heads of a group.  This file: the
// decode step, the token-by-token scan (f32, short portions, states too large for ssm_chunk.cu) and the gated norm behind
// all.  States, step sizes and decays are f32; a decay next to 1 enters as its difference from 1.
#include "dense_gemv.cuh"
#include "ssm.cuh"

namespace cera {

namespace {

constexpr int SS_WARPS = 8, SS_TILE = 16;

// grid (heads, slices of 32 values): lane = value, a warp takes every eighth row of the state.
template <class T>
__global__ void __launch_bounds__(SS_WARPS * 32) ssm_step_kernel(const float *pre, SsmView v, const uint32_t *pos_dev, float *y) {
    extern __shared__ float bc[];  // B, C of the head's group: [2][state_p]
    __shared__ float xs[32], part[SS_WARPS][32];
    const SsmShape &s = v.s;
    pdl_trigger();
    const uint32_t h = blockIdx.x, g = h / (s.heads / s.groups), p0 = blockIdx.y * 32, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, N = s.state_p;
    const float a_log = v.a_log[h], dt_bias = v.dt_bias[h], dd = v.d[h];
    pdl_wait();
    const uint32_t pos = *pos_dev, p = p0 + lane;
    float *S = v.state + ((size_t)h * N) * s.dim_p + p;
    constexpr int U = 16;
    float old[U];
    const bool live = p < s.dim_p;
#pragma unroll
    for (int k = 0; k < U; ++k) {
        const uint32_t r = warp + k * SS_WARPS;
        old[k] = live && r < N ? S[(size_t)r * s.dim_p] : 0.0f;
    }
    // the convolution: B and C of the group, x of the slice; the group's first head keeps the inputs of B and C, each slice its x
    const float *in = pre + s.inner_p();
    const bool keep_bc = blockIdx.y == 0 && h % (s.heads / s.groups) == 0;
    float *ring = v.conv.ring + (size_t)(pos % v.conv.taps) * v.conv.channels;
    for (uint32_t i = threadIdx.x; i < 2 * N + 32; i += SS_WARPS * 32) {
        const bool is_x = i >= 2 * N;
        if (is_x && p0 + i - 2 * N >= s.dim_p) continue;
        const uint32_t ch = is_x ? h * s.dim_p + p0 + i - 2 * N : i < N ? s.off_b() + g * N + i : s.off_c() + g * N + i - N;
        const float now = in[ch], val = Elem<T>::to(Elem<T>::from(silu_f32(conv_one(v.conv, ch, pos, now))));
        if (is_x) xs[i - 2 * N] = val;
        else bc[i] = val;
        if (is_x || keep_bc) ring[ch] = now;
    }
    const float dt = softplus_f32(pre[s.off_dt() + h] + dt_bias), am1 = expm1f(-expf(a_log) * dt);
    __syncthreads();
    const float x = live ? xs[lane] : 0.0f, dx = dt * x;
    float acc = 0.0f;
    for (uint32_t r0 = 0; r0 < N; r0 += U * SS_WARPS) {
        if (r0) {
#pragma unroll
            for (int k = 0; k < U; ++k) {
                const uint32_t r = r0 + warp + k * SS_WARPS;
                old[k] = live && r < N ? S[(size_t)r * s.dim_p] : 0.0f;
            }
        }
#pragma unroll
        for (int k = 0; k < U; ++k) {
            const uint32_t r = r0 + warp + k * SS_WARPS;
            if (r < N && live) {
                const float now = old[k] + fmaf(am1, old[k], bc[r] * dx);
                S[(size_t)r * s.dim_p] = now;
                acc = fmaf(now, bc[N + r], acc);
            }
        }
    }
    part[warp][lane] = acc;
    __syncthreads();
    if (warp == 0 && live) {
#pragma unroll
        for (int w = 1; w < SS_WARPS; ++w) acc += part[w][lane];
        y[(size_t)h * s.dim_p + p] = fmaf(dd, x, acc);
    }
}

// The same grid over a portion: the slice's state in shared memory, SS_TILE tokens' inputs at a time.
template <class T>
__global__ void __launch_bounds__(SS_WARPS * 32) ssm_scan_kernel(const float *pre, const T *xbc, SsmView v, uint32_t n, uint32_t start_pos, float *y) {
    extern __shared__ float sm[];
    __shared__ float xs[SS_TILE][32], dts[SS_TILE], as[SS_TILE], part[SS_TILE][SS_WARPS][32];
    const SsmShape &s = v.s;
    pdl_trigger();
    const uint32_t h = blockIdx.x, g = h / (s.heads / s.groups), p0 = blockIdx.y * 32, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, N = s.state_p;
    float *st = sm, *bs = st + (size_t)N * 32, *cs = bs + (size_t)SS_TILE * N;  // state [N][32], B and C [SS_TILE][N]
    const float a_log = v.a_log[h], dt_bias = v.dt_bias[h], dd = v.d[h];
    pdl_wait();
    const uint32_t p = p0 + lane;
    const bool live = p < s.dim_p;
    float *S = v.state + ((size_t)h * N) * s.dim_p + p;
    for (uint32_t r = warp; r < N; r += SS_WARPS) st[r * 32 + lane] = live ? S[(size_t)r * s.dim_p] : 0.0f;
    for (uint32_t t0 = 0; t0 < n; t0 += SS_TILE) {
        const uint32_t m = min((uint32_t)SS_TILE, n - t0);
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < m * N; i += SS_WARPS * 32) {
            const uint32_t t = i / N, r = i - t * N;
            const T *row = xbc + (size_t)(t0 + t) * s.channels();
            bs[i] = Elem<T>::to(row[s.off_b() + g * N + r]);
            cs[i] = Elem<T>::to(row[s.off_c() + g * N + r]);
        }
        for (uint32_t t = warp; t < m; t += SS_WARPS) {
            xs[t][lane] = live ? Elem<T>::to(xbc[(size_t)(t0 + t) * s.channels() + h * s.dim_p + p]) : 0.0f;
            if (lane == 0) {
                const float dt = softplus_f32(pre[(size_t)(t0 + t) * s.in_p + s.off_dt() + h] + dt_bias);
                dts[t] = dt;
                as[t] = expm1f(-expf(a_log) * dt);
            }
        }
        __syncthreads();
        for (uint32_t t = 0; t < m; ++t) {
            const float am1 = as[t], dx = dts[t] * xs[t][lane];
            float acc = 0.0f;
            for (uint32_t r = warp; r < N; r += SS_WARPS) {
                const float old = st[r * 32 + lane], now = old + fmaf(am1, old, bs[t * N + r] * dx);
                st[r * 32 + lane] = now;
                acc = fmaf(now, cs[t * N + r], acc);
            }
            part[t][warp][lane] = acc;
        }
        __syncthreads();
        for (uint32_t t = warp; t < m; t += SS_WARPS)
            if (live) {
                float acc = 0.0f;
#pragma unroll
                for (int w = 0; w < SS_WARPS; ++w) acc += part[t][w][lane];
                y[(size_t)(t0 + t) * s.inner_p() + h * s.dim_p + p] = fmaf(dd, xs[t][lane], acc);
            }
    }
    for (uint32_t r = warp; r < N; r += SS_WARPS)
        if (live) S[(size_t)r * s.dim_p] = st[r * 32 + lane];
    ssm_keep(pre, v, h, p0, min(p0 + 32, s.dim_p), blockIdx.y == 0, n, start_pos, SS_WARPS * 32);
}

constexpr int GN_KEEP = 8;  // values a thread holds in registers

// One CTA per (token, part).  Part g holds the model's own values [g * len, (g + 1) * len); head padding lies between them.
template <class T>
__global__ void __launch_bounds__(1024) gated_norm_kernel(const float *y, const float *pre, SsmView v, T *out, size_t ldo) {
    __shared__ float red[33];
    const SsmShape &s = v.s;
    pdl_trigger();
    pdl_wait();
    const uint32_t j = blockIdx.x, inner = s.heads * s.dim, len = inner / s.norm_groups, i0 = blockIdx.y * len, nt = blockDim.x;
    const float *yr = y + (size_t)j * s.inner_p(), *zr = pre + (size_t)j * s.in_p;
    float val[GN_KEEP], ss = 0.0f;
    auto at = [&](uint32_t i) { return s.dim == s.dim_p ? i : i / s.dim * s.dim_p + i % s.dim; };
    auto gated = [&](uint32_t i) {
        const uint32_t c = at(i);
        return yr[c] * silu_f32(zr[c]);
    };
#pragma unroll
    for (int k = 0; k < GN_KEEP; ++k) {
        const uint32_t i = threadIdx.x + k * nt;
        val[k] = i < len ? gated(i0 + i) : 0.0f;
        ss += val[k] * val[k];
    }
    for (uint32_t i = threadIdx.x + GN_KEEP * nt; i < len; i += nt) {
        const float x = gated(i0 + i);
        ss += x * x;
    }
    const float r = 1.0f / sqrtf(cta_sum(ss, red) / (float)len + s.eps);
    T *o = out + j * ldo;
#pragma unroll
    for (int k = 0; k < GN_KEEP; ++k) {
        const uint32_t i = threadIdx.x + k * nt;
        if (i < len) {
            const uint32_t c = at(i0 + i);
            o[c] = Elem<T>::from(val[k] * r * v.norm[c]);
        }
    }
    for (uint32_t i = threadIdx.x + GN_KEEP * nt; i < len; i += nt) {
        const uint32_t c = at(i0 + i);
        o[c] = Elem<T>::from(gated(i0 + i) * r * v.norm[c]);
    }
}

}  // namespace

int32_t launch_ssm_step(const float *pre, const SsmView &v, const uint32_t *pos_dev, float *y, int f32, cudaStream_t st) {
    const dim3 grid(v.s.heads, (v.s.dim_p + 31) / 32);
    count_launch();
    return gv::with_type(f32, [&](auto t) {
        return check_cuda(launch_k(ssm_step_kernel<decltype(t)>, grid, dim3(SS_WARPS * 32), (size_t)2 * v.s.state_p * 4, st, pre, v, pos_dev, y), "ssm step launch");
    });
}

int32_t launch_ssm_scan(const float *pre, const void *xbc, const SsmView &v, size_t n, size_t start_pos, float *y, int f32, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    const dim3 grid(v.s.heads, (v.s.dim_p + 31) / 32);
    const size_t smem = (size_t)v.s.state_p * (32 + 2 * SS_TILE) * 4;
    return gv::with_type(f32, [&](auto t) {
        using T = decltype(t);
        CERA_CUDA_TRY(cudaFuncSetAttribute(ssm_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, SSM_MAX_STATE * (32 + 2 * SS_TILE) * 4));
        count_launch();
        return check_cuda(launch_k(ssm_scan_kernel<T>, grid, dim3(SS_WARPS * 32), smem, st, pre, (const T *)xbc, v, (uint32_t)n, (uint32_t)start_pos, y), "ssm scan launch");
    });
}

int32_t launch_gated_norm(const float *y, const float *pre, const SsmView &v, size_t n, void *out, size_t ldo, int f32, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    const dim3 grid((unsigned)n, v.s.norm_groups);
    const uint32_t len = v.s.heads * v.s.dim / v.s.norm_groups;
    uint32_t threads = 64;
    while (threads < 1024 && threads * (n == 1 ? 2 : GN_KEEP) < len) threads *= 2;
    count_launch();
    return gv::with_type(f32, [&](auto t) {
        using T = decltype(t);
        return check_cuda(launch_k(gated_norm_kernel<T>, grid, dim3(threads), 0, st, y, pre, v, (T *)out, ldo), "gated norm launch");
    });
}

}  // namespace cera
