// Many-column products with dense weights on the CUDA cores (f32 FMA): the f32 path, and bf16 shapes the tcgen05 kernel
// (dense_gemm_tc.cu) does not take.  64 x 64 tiles, 16 k-elements per step.
#include "dense.cuh"

namespace cera {

namespace {

constexpr int GM_TILE = 64, GM_K = 16;

template <class T>
__global__ void __launch_bounds__(256) dense_gemm_kernel(DenseGemm g) {
    __shared__ float ws[GM_K][GM_TILE + 4], xs[GM_K][GM_TILE + 4];
    pdl_trigger();
    pdl_wait();
    uint32_t row_base = 0, rows = g.w.rows, first = blockIdx.y * GM_TILE, end = g.n;
    if (g.tiles) {  // blockIdx.y walks (item, 64-column part)
        const uint32_t parts = (g.group_columns + GM_TILE - 1) / GM_TILE, item = blockIdx.y / parts;
        if (item >= *g.n_tiles) return;
        const MoeTile t = g.tiles[item];
        row_base = t.expert * g.rows_per_expert;
        rows = g.rows_per_expert;
        first = t.first + (blockIdx.y % parts) * GM_TILE;
        end = t.first + t.count;
        if (first >= end) return;
    }
    const uint32_t r0 = blockIdx.x * GM_TILE, ld = g.w.ld, xld = g.x_ld ? g.x_ld : ld;
    const T *w = (const T *)g.w.w + (size_t)row_base * ld, *x = (const T *)g.x + (g.block_rows ? (size_t)(r0 / g.block_rows) * ld : 0);
    const uint32_t tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < ld; k0 += GM_K) {
        for (uint32_t i = threadIdx.x; i < GM_TILE * GM_K; i += 256) {
            const uint32_t r = i / GM_K, k = i % GM_K;
            ws[k][r] = r0 + r < rows ? Elem<T>::to(w[(size_t)(r0 + r) * ld + k0 + k]) : 0.0f;
            xs[k][r] = first + r < end ? Elem<T>::to(x[(size_t)(first + r) * xld + k0 + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < GM_K; ++k) {
            const float4 a = *reinterpret_cast<const float4 *>(&ws[k][tx * 4]), b = *reinterpret_cast<const float4 *>(&xs[k][ty * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const uint32_t col = first + ty * 4 + j;
        if (col >= end) continue;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const uint32_t row = r0 + tx * 4 + i;
            if (row >= rows) continue;
            if (g.out_kind == DENSE_F32) ((float *)g.out)[(size_t)col * g.ldo + row] = acc[i][j];
            else if (g.out_kind == DENSE_T) ((T *)g.out)[(size_t)col * g.ldo + row] = Elem<T>::from(acc[i][j]);
            else ((T *)g.out)[(size_t)row * g.ldo + col] = Elem<T>::from(acc[i][j]);
        }
    }
}

// The gated unit over columns: pre [n][2 ff_p] -> out [n][ff_p].
template <class T>
__global__ void __launch_bounds__(256) gated_unit_kernel(const float *pre, uint32_t n, uint32_t ff_p, const float *col_scale, ExpertAct a, T *out) {
    pdl_trigger();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= (size_t)n * ff_p) return;
    const uint32_t j = (uint32_t)(i / ff_p), f = (uint32_t)(i - (size_t)j * ff_p);
    const float s = col_scale ? col_scale[j] : 1.0f;
    out[i] = Elem<T>::from(gated_unit(s * pre[(size_t)j * 2 * ff_p + f], s * pre[(size_t)j * 2 * ff_p + ff_p + f], a));
}

}  // namespace

int32_t launch_dense_gemm(const DenseGemm &g, cudaStream_t st) {
    if (g.n == 0) return CERA_CUDA_OK;
    bool taken = false;
    if (!g.w.f32) CERA_TRY(launch_dense_gemm_tc(g, st, &taken));
    if (taken) return CERA_CUDA_OK;
    if (g.out_kind == DENSE_GATED_UNIT) {
        // the products into a stream-ordered scratch, then the unit
        const uint32_t ff_p = (g.tiles ? g.rows_per_expert : g.w.rows) / 2;
        float *pre = nullptr;
        CERA_CUDA_TRY(cudaMallocAsync((void **)&pre, (size_t)g.n * 2 * ff_p * 4, st));
        DenseGemm p = g;
        p.out_kind = DENSE_F32;
        p.out = pre;
        p.ldo = 2 * ff_p;
        int32_t rc = launch_dense_gemm(p, st);
        if (rc == CERA_CUDA_OK) {
            const unsigned grid = (unsigned)(((size_t)g.n * ff_p + 255) / 256);
            count_launch();
            rc = check_cuda(g.w.f32 ? launch_k(gated_unit_kernel<float>, dim3(grid), dim3(256), 0, st, (const float *)pre, g.n, ff_p, g.col_scale, g.act, (float *)g.out)
                                    : launch_k(gated_unit_kernel<bf16>, dim3(grid), dim3(256), 0, st, (const float *)pre, g.n, ff_p, g.col_scale, g.act, (bf16 *)g.out),
                            "gated unit launch");
        }
        const cudaError_t e = cudaFreeAsync(pre, st);
        CERA_TRY(rc);
        return check_cuda(e, "cudaFreeAsync(gated unit)");
    }
    const uint32_t rows = g.tiles ? g.rows_per_expert : g.w.rows;
    const dim3 grid((rows + GM_TILE - 1) / GM_TILE, g.tiles ? g.max_tiles * ((g.group_columns + GM_TILE - 1) / GM_TILE) : (g.n + GM_TILE - 1) / GM_TILE);
    count_launch();
    return check_cuda(g.w.f32 ? launch_k(dense_gemm_kernel<float>, grid, dim3(256), 0, st, g) : launch_k(dense_gemm_kernel<bf16>, grid, dim3(256), 0, st, g),
                      "dense gemm launch");
}

}  // namespace cera
