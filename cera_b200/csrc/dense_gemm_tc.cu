// Many-column bf16 products on the fifth-generation tensor cores: out[column][row] = W x, tcgen05.mma kind::f16 with f32
// accumulators in TMEM.  A persistent CTA walks output tiles of 128 weight rows x BN columns (tokens): one thread keeps a
// ring of stages filled by TMA (64 elements of k, 128-byte swizzle), one thread issues the MMAs, eight warps drain the
// finished accumulator - lane = weight row, so a column's values leave as consecutive stores; two warps share 32 rows and
// take 32 columns in turn - while the next tile's MMAs run into the other accumulator.
//
// Grouped by expert the tiles come from a device-built work list.  With NA = 2 a stage holds two weight tiles (an expert's
// gate rows and the same up rows; without groups, the matrix's first and second half) against one activation tile, and the
// epilogue forms the gated unit from the two accumulators.  Every wait is bounded (tma.cuh); a wait that runs out empties the CTA and raises a status bit.
#include <cudaTypedefs.h>

#include "dense.cuh"
#include "tc.cuh"
#include "tensor_map.h"

namespace cera {

__device__ unsigned int g_dense_tc_status = 0;

// bits 17..19: roles of this kernel (loader, MMA, epilogue); bits 20..22: the prompt attention's (attention_tc.cu)
static const bool g_dense_tc_registered = register_kernel_status([] {
    unsigned int v = 0;
    cudaMemcpyFromSymbol(&v, g_dense_tc_status, sizeof(v));
    return (uint32_t)v << 17;
});

int32_t tensor_map_bf16(CUtensorMap *map, const void *base, uint64_t rows, uint64_t ld, uint32_t box_cols, uint32_t box_rows) {
    static PFN_cuTensorMapEncodeTiled_v12000 encode = [] {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &p, 12000, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
            p = nullptr;
        return (PFN_cuTensorMapEncodeTiled_v12000)p;
    }();
    if (!encode) return fail(CERA_CUDA_ERR_CUDA, "the driver offers no cuTensorMapEncodeTiled");
    const cuuint64_t dims[2] = {ld, rows}, strides[1] = {ld * 2};
    const cuuint32_t box[2] = {box_cols, box_rows}, es[2] = {1, 1};
    const CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(CERA_CUDA_ERR_CUDA, "cuTensorMapEncodeTiled: error %d for [%llu x %llu]", (int)r, (unsigned long long)rows, (unsigned long long)ld);
    return CERA_CUDA_OK;
}

namespace {

constexpr int DT_BM = 128, DT_KS = 64, DT_THREADS = 10 * 32;  // loader, MMA, eight epilogue warps
constexpr uint32_t DT_A_BYTES = DT_BM * DT_KS * 2;

template <int BN, int NA>
struct Tile {
    static constexpr uint32_t B_BYTES = BN * DT_KS * 2, STAGE = NA * DT_A_BYTES + B_BYTES;
    static constexpr int STAGES = 200 * 1024 / STAGE < 8 ? 200 * 1024 / STAGE : 8;
    static constexpr uint32_t ACC = NA * BN, COLS = 2 * ACC;  // TMEM columns of one accumulator, of both
    static constexpr uint32_t TMEM = COLS <= 64 ? 64 : COLS <= 128 ? 128 : COLS <= 256 ? 256 : 512;
    static constexpr uint32_t SMEM = STAGES * STAGE + 1024 + 256;
};

struct DtParams {
    DenseGemm g;
    uint32_t row_tiles, col_tiles;
};

// Output tile t of this launch.
struct DtTile {
    uint32_t a_row, row0, rows, first, end;
};
template <int BN, int NA>
__device__ __forceinline__ DtTile dt_tile(const DtParams &p, uint32_t t) {
    DtTile o;
    if (p.g.tiles) {
        const MoeTile m = p.g.tiles[t / p.row_tiles];
        o.row0 = (t % p.row_tiles) * DT_BM;
        o.rows = NA == 2 ? p.g.rows_per_expert / 2 : p.g.rows_per_expert;
        o.a_row = m.expert * p.g.rows_per_expert + o.row0;
        o.first = m.first;
        o.end = m.first + m.count;
    } else {
        o.row0 = o.a_row = (t / p.col_tiles) * DT_BM;
        o.rows = p.g.w.rows / NA;
        o.first = (t % p.col_tiles) * BN;
        o.end = min(o.first + BN, p.g.n);
    }
    return o;
}

template <int BN, int NA>
__global__ void __launch_bounds__(DT_THREADS, 1) dense_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, DtParams p) {
    using S = Tile<BN, NA>;
    extern __shared__ uint8_t raw[];
    uint8_t *stages = raw + (1024 - (tma::smem_u32(raw) & 1023)) % 1024;
    uint64_t *full = reinterpret_cast<uint64_t *>(stages + S::STAGES * S::STAGE), *empty = full + S::STAGES, *acc_full = empty + S::STAGES, *acc_empty = acc_full + 2;
    uint32_t *tmem_at = reinterpret_cast<uint32_t *>(acc_empty + 2);
    volatile uint32_t *abort_flag = tmem_at + 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    if (threadIdx.x == 0) {
        for (int i = 0; i < S::STAGES; ++i) {
            tma::mbar_init(full + i, 1);
            tma::mbar_init(empty + i, 1);
        }
        for (int i = 0; i < 2; ++i) {
            tma::mbar_init(acc_full + i, 1);
            tma::mbar_init(acc_empty + i, 8);
        }
        *abort_flag = 0;
        tma::mbar_init_fence();
    }
    if (warp == 1) {
        tmem_alloc(tmem_at, S::TMEM);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_at;
    pdl_wait();
    const uint32_t n_tiles = p.g.tiles ? *p.g.n_tiles * p.row_tiles : p.row_tiles * p.col_tiles, n_k = p.g.w.ld / DT_KS;
    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            bool ok = true;
            for (uint32_t t = blockIdx.x; t < n_tiles && ok; t += gridDim.x) {
                const DtTile o = dt_tile<BN, NA>(p, t);
                const uint32_t x0 = p.g.block_rows ? o.a_row / p.g.block_rows * p.g.w.ld : 0;
                for (uint32_t k = 0; k < n_k; ++k, ++it) {
                    const uint32_t s = it % S::STAGES;
                    if (!(ok = tma::mbar_wait_blocking(empty + s, (it / S::STAGES & 1) ^ 1, abort_flag, &g_dense_tc_status, 1u))) break;
                    uint8_t *st = stages + s * S::STAGE;
                    tma::mbar_expect_tx(full + s, S::STAGE);
                    tma::tensor_g2s_2d(st, &map_w, k * DT_KS, o.a_row, full + s);
                    if (NA == 2) tma::tensor_g2s_2d(st + DT_A_BYTES, &map_w, k * DT_KS, o.a_row + o.rows, full + s);
                    tma::tensor_g2s_2d(st + NA * DT_A_BYTES, &map_x, x0 + k * DT_KS, o.first, full + s);
                }
            }
            // given up: this CTA's shared memory must outlive the copies in flight
            if (*abort_flag)
                for (uint32_t i = it > S::STAGES ? it - S::STAGES : 0; i < it; ++i)
                    for (uint32_t n = 0; n < tma::SPIN_LIMIT && !tma::mbar_test(full + i % S::STAGES, i / S::STAGES & 1); ++n) __nanosleep(40);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t it = 0, j = 0;
            bool ok = true;
            for (uint32_t t = blockIdx.x; t < n_tiles && ok; t += gridDim.x, ++j) {
                const uint32_t b = j & 1, acc = tmem + b * S::ACC;
                if (!(ok = tma::mbar_wait_blocking(acc_empty + b, (j >> 1 & 1) ^ 1, abort_flag, &g_dense_tc_status, 2u))) break;
                tc_fence_after();
                for (uint32_t k = 0; k < n_k; ++k, ++it) {
                    const uint32_t s = it % S::STAGES;
                    if (!(ok = tma::mbar_wait_blocking(full + s, it / S::STAGES & 1, abort_flag, &g_dense_tc_status, 2u))) break;
                    tc_fence_after();
                    const uint32_t st = tma::smem_u32(stages + s * S::STAGE);
                    const uint64_t da = smem_desc_sw128(st), db = smem_desc_sw128(st + NA * DT_A_BYTES);
#pragma unroll
                    for (int kk = 0; kk < DT_KS / 16; ++kk) {
                        tc_mma_f16(acc, da + 2 * kk, db + 2 * kk, tc_idesc_bf16(DT_BM, BN), k | kk);
                        if (NA == 2) tc_mma_f16(acc + BN, smem_desc_sw128(st + DT_A_BYTES) + 2 * kk, db + 2 * kk, tc_idesc_bf16(DT_BM, BN), k | kk);
                    }
                    tc_commit(empty + s);
                }
                if (ok) tc_commit(acc_full + b);
            }
        }
    } else {
        const uint32_t quad = warp & 3;  // the TMEM lanes this warp may read: [32 quad, + 32)
        const uint32_t turn = (warp - 2) >> 2;
        uint32_t j = 0;
        for (uint32_t t = blockIdx.x; t < n_tiles; t += gridDim.x, ++j) {
            const uint32_t b = j & 1;
            const bool ok = tma::mbar_wait_blocking(acc_full + b, j >> 1 & 1, abort_flag, &g_dense_tc_status, 4u);
            if (!__all_sync(0xffffffffu, ok)) break;
            tc_fence_after();
            const DtTile o = dt_tile<BN, NA>(p, t);
            const uint32_t row = o.row0 + quad * 32 + lane, acc = tmem + b * S::ACC + (quad * 32 << 16), cols = o.end - o.first;
            const bool live = row < o.rows;
#pragma unroll 1
            for (uint32_t c0 = turn * 32; c0 < BN && c0 < cols; c0 += 64) {
                uint32_t v[2][16];
                tmem_ld16(acc + c0, v[0]);
                tmem_ld16(acc + c0 + 16, v[1]);
                if (NA == 2) {
                    uint32_t u[2][16];
                    tmem_ld16(acc + BN + c0, u[0]);
                    tmem_ld16(acc + BN + c0 + 16, u[1]);
                    tmem_wait_ld();
#pragma unroll
                    for (int c = 0; c < 32; ++c) {
                        const uint32_t col = o.first + c0 + c;
                        if (live && col < o.end) {
                            const float sc = p.g.col_scale ? p.g.col_scale[col] : 1.0f;
                            ((bf16 *)p.g.out)[(size_t)col * p.g.ldo + row] = __float2bfloat16_rn(
                                gated_unit(sc * __uint_as_float(v[c >> 4][c & 15]), sc * __uint_as_float(u[c >> 4][c & 15]), p.g.act));
                        }
                    }
                    continue;
                }
                tmem_wait_ld();
                if (p.g.out_kind == DENSE_F32) {
                    float *out = (float *)p.g.out + (size_t)(o.first + c0) * p.g.ldo + row;
#pragma unroll
                    for (int c = 0; c < 32; ++c)
                        if (live && c0 + c < cols) out[(size_t)c * p.g.ldo] = __uint_as_float(v[c >> 4][c & 15]);
                } else if (p.g.out_kind == DENSE_T) {
                    bf16 *out = (bf16 *)p.g.out + (size_t)(o.first + c0) * p.g.ldo + row;
#pragma unroll
                    for (int c = 0; c < 32; ++c)
                        if (live && c0 + c < cols) out[(size_t)c * p.g.ldo] = __float2bfloat16_rn(__uint_as_float(v[c >> 4][c & 15]));
                } else if (live) {  // transposed: 32 consecutive columns of this row; columns past the end are zeros of the operand
                    uint4 *out = reinterpret_cast<uint4 *>((bf16 *)p.g.out + (size_t)row * p.g.ldo + o.first + c0);
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        uint32_t w[4];
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            const int c = q * 8 + i * 2;
                            const __nv_bfloat162 pr = __floats2bfloat162_rn(__uint_as_float(v[c >> 4][c & 15]), __uint_as_float(v[c >> 4][(c & 15) + 1]));
                            w[i] = *reinterpret_cast<const uint32_t *>(&pr);
                        }
                        if (o.first + c0 + q * 8 + 8 <= p.g.ldo) out[q] = make_uint4(w[0], w[1], w[2], w[3]);
                    }
                }
            }
            tc_fence_before();
            if (lane == 0) tma::mbar_arrive(acc_empty + b);
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, S::TMEM);
}

template <int BN, int NA>
int32_t launch_tc(const DenseGemm &g, cudaStream_t st) {
    using S = Tile<BN, NA>;
    CUtensorMap mw, mx;
    CERA_TRY(tensor_map_bf16(&mw, g.w.w, g.w.rows, g.w.ld, DT_KS, DT_BM));
    CERA_TRY(tensor_map_bf16(&mx, g.x, g.n, g.row_len(), DT_KS, BN));
    DtParams p;
    p.g = g;
    const uint32_t rows = (g.tiles ? g.rows_per_expert : g.w.rows) / NA;
    p.row_tiles = (rows + DT_BM - 1) / DT_BM;
    p.col_tiles = g.tiles ? g.max_tiles : (g.n + BN - 1) / BN;
    const uint64_t tiles = (uint64_t)p.row_tiles * p.col_tiles;
    const unsigned grid = tiles < (uint64_t)sm_count() ? (unsigned)tiles : (unsigned)sm_count();
    auto k = dense_gemm_tc_kernel<BN, NA>;
    CERA_CUDA_TRY(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, S::SMEM));
    count_launch();
    return check_cuda(launch_k(k, dim3(grid), dim3(DT_THREADS), S::SMEM, st, mw, mx, p), "dense tcgen05 gemm launch");
}

}  // namespace

int32_t launch_dense_gemm_tc(const DenseGemm &g, cudaStream_t st, bool *taken) {
    *taken = false;
    if (g.w.f32 || g.w.ld % DT_KS || g.n == 0) return CERA_CUDA_OK;
    if (g.out_kind == DENSE_T_TRANSPOSED && g.ldo % 8) return CERA_CUDA_OK;
    *taken = true;
    const bool pair = g.out_kind == DENSE_GATED_UNIT;
    if (g.tiles) {
        if (g.group_columns <= 32) return pair ? launch_tc<32, 2>(g, st) : launch_tc<32, 1>(g, st);
        if (g.group_columns <= 64) return pair ? launch_tc<64, 2>(g, st) : launch_tc<64, 1>(g, st);
        return pair ? launch_tc<128, 2>(g, st) : launch_tc<128, 1>(g, st);
    }
    if (pair) return g.n <= 32 ? launch_tc<32, 2>(g, st) : g.n <= 64 ? launch_tc<64, 2>(g, st) : launch_tc<128, 2>(g, st);
    const uint32_t row_tiles = (g.w.rows + DT_BM - 1) / DT_BM;
    if (g.n <= 32) return launch_tc<32, 1>(g, st);
    if (g.n <= 64) return launch_tc<64, 1>(g, st);
    if (g.n <= 128 || row_tiles * ((g.n + 255) / 256) < (uint32_t)sm_count() * 3 / 4) return launch_tc<128, 1>(g, st);
    return launch_tc<256, 1>(g, st);
}

}  // namespace cera
