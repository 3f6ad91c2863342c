// Weight placement, embedding and sublayer boundaries of models described layer by layer.
#include <cuda_fp16.h>

#include "dense.cuh"
#include "model.h"

namespace cera {

namespace {

__device__ __forceinline__ float load_src(const void *p, int type, size_t i) {
    if (type == CERA_TYPE_F32) return ((const float *)p)[i];
    if (type == CERA_TYPE_F16) return __half2float(((const __half *)p)[i]);
    return __bfloat162float(((const bf16 *)p)[i]);
}

__global__ void place_kernel(const void *__restrict__ src, int type, size_t rows, uint32_t cols, void *dst, int dst_f32, size_t ld, PadMap rmap,
                             PadMap cmap, float offset) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= rows * cols) return;
    const uint32_t r = (uint32_t)(i / cols), c = (uint32_t)(i - (size_t)r * cols);
    const size_t o = (size_t)rmap(r) * ld + cmap(c);
    const float v = load_src(src, type, i) + offset;
    if (dst_f32) ((float *)dst)[o] = v;
    else ((bf16 *)dst)[o] = __float2bfloat16_rn(v);
}

template <class T>
__global__ void __launch_bounds__(256) embed_dense_kernel(const T *__restrict__ table, const T *__restrict__ bigram, BigramParams bp, uint32_t ld,
                                                          const uint32_t *tokens, const uint32_t *dyn, float scale, float *x, float *keep) {
    pdl_trigger();
    pdl_wait();
    const uint32_t j = blockIdx.y;
    const uint32_t tok = dyn ? dyn[DYN_TOKEN] : tokens[j + 1], prev = dyn ? dyn[DYN_PREV] : tokens[j];
    const T *row = table + (size_t)tok * ld;
    const T *brow = nullptr;
    if (bp.buckets) {
        const uint64_t b = prev == NO_TOKEN ? bp.buckets : (prev * bp.mul_prev + tok * bp.mul_cur) % bp.buckets;
        brow = bigram + (size_t)b * ld;
    }
    for (uint32_t i = blockIdx.x * blockDim.x + threadIdx.x; i < ld; i += gridDim.x * blockDim.x) {
        float v = Elem<T>::to(row[i]) * scale;
        if (brow) v += Elem<T>::to(brow[i]);
        x[(size_t)j * ld + i] = v;
        if (keep) keep[(size_t)j * ld + i] = v;
    }
}

// One CTA per row, four numbers per thread and vector, the row in registers (V vectors a thread).  The padding of x and y
// is zero, so whole vectors are summed.
template <class T, int V>
__global__ void __launch_bounds__(1024) residual_norm_kernel(ResidualNorm p, uint32_t width, uint32_t ld, float eps) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const uint32_t j = blockIdx.x, t = threadIdx.x, nt = blockDim.x, nv = ld / 4;
    float4 *x = reinterpret_cast<float4 *>(p.x + (size_t)(p.x_rows ? p.x_rows[j] : j) * ld);
    const float inv_w = 1.0f / (float)width;
    float4 xv[V], yv[V];
    float ss = 0.0f;
#pragma unroll
    for (int e = 0; e < V; ++e) {
        const uint32_t i = t + e * nt;
        xv[e] = yv[e] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (i < nv) {
            xv[e] = x[i];
            if (p.y && !p.entry_of) yv[e] = reinterpret_cast<const float4 *>(p.y + (size_t)j * ld)[i];
        }
    }
    if (p.y) {
        if (p.entry_of) {
            for (uint32_t s = 0; s < p.picks; ++s) {
                const float4 *row = reinterpret_cast<const float4 *>(p.y + (size_t)p.entry_of[j * p.picks + s] * ld);
                const float w = p.pick_weight ? p.pick_weight[j * p.picks + s] : 1.0f;
#pragma unroll
                for (int e = 0; e < V; ++e)
                    if (t + e * nt < nv) {
                        const float4 r = row[t + e * nt];
                        yv[e].x += w * r.x;
                        yv[e].y += w * r.y;
                        yv[e].z += w * r.z;
                        yv[e].w += w * r.w;
                    }
            }
        }
        float r = 1.0f;
        if (p.post.g) {
#pragma unroll
            for (int e = 0; e < V; ++e) ss += yv[e].x * yv[e].x + yv[e].y * yv[e].y + yv[e].z * yv[e].z + yv[e].w * yv[e].w;
            r = 1.0f / sqrtf(cta_sum(ss, red) * inv_w + eps);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const uint32_t i = t + e * nt;
            if (i < nv) {
                const float4 g = p.post.g ? p.post.at(i) : make_float4(1.0f, 1.0f, 1.0f, 1.0f);
                xv[e].x += yv[e].x * r * g.x;
                xv[e].y += yv[e].y * r * g.y;
                xv[e].z += yv[e].z * r * g.z;
                xv[e].w += yv[e].w * r * g.w;
            }
        }
        ss = 0.0f;
    }
    if (p.y || p.add) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const uint32_t i = t + e * nt;
            if (i >= nv) continue;
            if (p.add) {
                const float4 a = reinterpret_cast<const float4 *>(p.add + (size_t)j * ld)[i];
                xv[e].x += a.x;
                xv[e].y += a.y;
                xv[e].z += a.z;
                xv[e].w += a.w;
            }
            x[i] = xv[e];
        }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) ss += xv[e].x * xv[e].x + xv[e].y * xv[e].y + xv[e].z * xv[e].z + xv[e].w * xv[e].w;
    const float r = 1.0f / sqrtf(cta_sum(ss, red) * inv_w + eps);
#pragma unroll
    for (int e = 0; e < V; ++e) {
        const uint32_t i = t + e * nt;
        if (i >= nv) continue;
        const float4 g = p.pre.at(i);
        const float4 v = make_float4(xv[e].x * r * g.x, xv[e].y * r * g.y, xv[e].z * r * g.z, xv[e].w * r * g.w);
        if (p.h) store4((T *)p.h + (size_t)j * ld + 4 * i, v);
        if (p.h32) reinterpret_cast<float4 *>(p.h32 + (size_t)j * ld)[i] = v;
    }
}

// One CTA per (token, pick): the next place in the expert's bucket, and the token's row there.
__global__ void __launch_bounds__(128) moe_gather_kernel(const uint4 *h, uint32_t row_vecs, const uint32_t *ids,
                                                         const float *weights, uint32_t n_used, uint32_t *cursor, uint32_t *entry_of,
                                                         uint4 *g, float *col_scale) {
    __shared__ uint32_t pos_s;
    pdl_trigger();
    pdl_wait();
    const uint32_t pair = blockIdx.x, j = pair / n_used;
    if (threadIdx.x == 0) {
        pos_s = atomicAdd(cursor + ids[pair], 1u);
        entry_of[pair] = pos_s;
        col_scale[pos_s] = weights[pair];
    }
    __syncthreads();
    const size_t pos = pos_s;
    for (uint32_t i = threadIdx.x; i < row_vecs; i += blockDim.x) g[pos * row_vecs + i] = h[(size_t)j * row_vecs + i];
}

}  // namespace

int32_t launch_place(const void *src, int32_t src_type, size_t rows, size_t cols, void *dst, int dst_f32, size_t ld, const PadMap &rmap,
                     const PadMap &cmap, cudaStream_t st, float offset) {
    if (src_type != CERA_TYPE_F32 && src_type != CERA_TYPE_F16 && src_type != CERA_TYPE_BF16)
        return fail(CERA_CUDA_ERR_UNSUPPORTED, "dense weight: ggml type %d is not F32, F16 or BF16", src_type);
    const size_t total = rows * cols;
    if (total == 0) return CERA_CUDA_OK;
    place_kernel<<<(unsigned)((total + 255) / 256), 256, 0, st>>>(src, src_type, rows, (uint32_t)cols, dst, dst_f32, ld, rmap, cmap, offset);
    count_launch();
    return check_cuda(cudaGetLastError(), "place launch");
}

int32_t launch_embed_dense(const DenseView &table, const DenseView &bigram, const BigramParams &bp, const uint32_t *tokens, const uint32_t *dyn,
                           size_t n, float scale, float *x, float *keep, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    const dim3 grid((table.ld + 1023) / 1024, (unsigned)n);
    count_launch();
    if (table.f32)
        return check_cuda(launch_k(embed_dense_kernel<float>, grid, dim3(256), 0, st, (const float *)table.w, (const float *)bigram.w, bp, table.ld,
                                   tokens, dyn, scale, x, keep), "embed launch");
    return check_cuda(launch_k(embed_dense_kernel<bf16>, grid, dim3(256), 0, st, (const bf16 *)table.w, (const bf16 *)bigram.w, bp, table.ld, tokens,
                               dyn, scale, x, keep), "embed launch");
}

int32_t launch_residual_norm(const ResidualNorm &p, uint32_t width, uint32_t ld, size_t n, float eps, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    const uint32_t nv = ld / 4;
    // one vector a thread for a lone row, four for many
    uint32_t v = n == 1 ? 1 : 4;
    while (v > 1 && nv < v * 32) v /= 2;
    while (v < 16 && (nv + v - 1) / v > 1024) v *= 2;
    const uint32_t threads = ((nv + v - 1) / v + 31) / 32 * 32;
    if (threads > 1024) return fail(CERA_CUDA_ERR_UNSUPPORTED, "norm: rows of %u numbers (at most 65536)", width);
    auto go = [&](auto kernel) {
        count_launch();
        return check_cuda(launch_k(kernel, dim3((unsigned)n), dim3(threads), 0, st, p, width, ld, eps), "residual norm launch");
    };
    auto typed = [&](auto t) {
        using T = decltype(t);
        switch (v) {
            case 1: return go(residual_norm_kernel<T, 1>);
            case 2: return go(residual_norm_kernel<T, 2>);
            case 4: return go(residual_norm_kernel<T, 4>);
            case 8: return go(residual_norm_kernel<T, 8>);
            default: return go(residual_norm_kernel<T, 16>);
        }
    };
    return p.h_f32 ? typed(float{}) : typed(bf16{});
}

int32_t launch_moe_gather(const void *h, int f32, uint32_t ld, const uint32_t *ids, const float *weights, uint32_t n_used, size_t n, uint32_t *cursor,
                          uint32_t *entry_of, void *g, float *col_scale, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    count_launch();
    return check_cuda(launch_k(moe_gather_kernel, dim3((unsigned)(n * n_used)), dim3(128), 0, st, (const uint4 *)h, ld * (f32 ? 4 : 2) / 16, ids, weights,
                               n_used, cursor, entry_of, (uint4 *)g, col_scale),
                      "moe gather launch");
}

}  // namespace cera
