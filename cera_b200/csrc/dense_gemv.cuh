// Building blocks of the one-column products: a row group (R rows that share the activation vector) is walked by WPR warps
// of a CTA, 16 bytes per lane and row at a time; the first loads are issued before the kernel waits for its predecessor
// (weights never change).
#pragma once

#include "dense.cuh"

namespace cera {

namespace gv {

constexpr int GV_WARPS = 8;

template <class T, int R, int U>
struct RowDot {
    const T *w[R];
    uint32_t nv, step, c;
    uint4 buf[R][U];
    // part of `parts` warps that share the row; ld elements per row
    __device__ __forceinline__ void start(uint32_t ld, int part, int parts) {
        nv = ld / Elem<T>::N;
        step = 32u * parts;
        c = part * 32u + (threadIdx.x & 31);
    }
    __device__ __forceinline__ void fetch() {
#pragma unroll
        for (int u = 0; u < U; ++u)
            if (c + u * step < nv) {
#pragma unroll
                for (int r = 0; r < R; ++r) buf[r][u] = ld_stream(reinterpret_cast<const uint4 *>(w[r]) + c + u * step);
            }
    }
    __device__ __forceinline__ void run(const T *x, float (&acc)[R]) {
        while (c < nv) {
#pragma unroll
            for (int u = 0; u < U; ++u)
                if (c + u * step < nv) {
                    float xf[Elem<T>::N], wf[Elem<T>::N];
                    Elem<T>::unpack(*(reinterpret_cast<const uint4 *>(x) + c + u * step), xf);
#pragma unroll
                    for (int r = 0; r < R; ++r) {
                        Elem<T>::unpack(buf[r][u], wf);
#pragma unroll
                        for (int i = 0; i < Elem<T>::N; ++i) acc[r] = fmaf(wf[i], xf[i], acc[r]);
                    }
                }
            c += U * step;
            fetch();
        }
    }
};

// Sums of R values over the WPR warps of a group; valid in lane 0 of the group's first warp.
template <int R, int WPR>
__device__ __forceinline__ void group_sum(float (&acc)[R], float (*red)[R]) {
#pragma unroll
    for (int r = 0; r < R; ++r) acc[r] = warp_sum(acc[r]);
    if (WPR == 1) return;
    const int warp = threadIdx.x >> 5;
    if ((threadIdx.x & 31) == 0) {
#pragma unroll
        for (int r = 0; r < R; ++r) red[warp][r] = acc[r];
    }
    __syncthreads();
    if (warp % WPR == 0) {
#pragma unroll
        for (int r = 0; r < R; ++r) {
            acc[r] = 0.0f;
#pragma unroll
            for (int i = 0; i < WPR; ++i) acc[r] += red[warp + i][r];
        }
    }
}

// Warps per row group: shared further while every warp keeps a batch of loads (u vectors a lane) and all groups still run
// at once; few groups are shared whatever the batch.
inline int pick_wpr(size_t groups, size_t row_bytes, int u) {
    const size_t vecs = row_bytes / 16, few = (size_t)sm_count() * 14, room = (size_t)sm_count() * 64;
    int wpr = 1;
    while (wpr < 8 && (groups * wpr < few || (groups * wpr * 2 <= room && vecs >= (size_t)wpr * 2 * 32 * u))) wpr *= 2;
    return wpr;
}

template <class F>
int32_t with_wpr(int wpr, F f) {
    switch (wpr) {
        case 1: return f(std::integral_constant<int, 1>{});
        case 2: return f(std::integral_constant<int, 2>{});
        case 4: return f(std::integral_constant<int, 4>{});
        default: return f(std::integral_constant<int, 8>{});
    }
}
template <class F>
int32_t with_type(int f32, F f) {
    return f32 ? f(float{}) : f(bf16{});
}
inline dim3 gv_grid(size_t groups, int wpr, uint32_t y = 1) { return dim3((unsigned)((groups * wpr + GV_WARPS - 1) / GV_WARPS), y); }

}  // namespace gv

}  // namespace cera
