// One-column products with dense weights: the decode step's projections, with the work that follows them fused where
// one warp holds all a result needs (the minGRU update, the gated units, the sum over picks).
#include "dense_gemv.cuh"
#include "moe_route.cuh"

namespace cera {

namespace {

using namespace gv;

template <class T, int R, int WPR>
__global__ void __launch_bounds__(GV_WARPS * 32) gemv_kernel(const T *__restrict__ w, uint32_t rows, uint32_t ld, const T *x, float *y) {
    __shared__ float red[GV_WARPS][R];
    pdl_trigger();
    const int warp = threadIdx.x >> 5;
    const uint32_t g = blockIdx.x * (GV_WARPS / WPR) + warp / WPR;
    RowDot<T, R, R == 1 ? 8 : 4> d;
#pragma unroll
    for (int r = 0; r < R; ++r) d.w[r] = w + (size_t)min(g * R + r, rows - 1) * ld;
    d.start(ld, warp % WPR, WPR);
    d.fetch();
    pdl_wait();
    float acc[R] = {};
    d.run(x, acc);
    group_sum<R, WPR>(acc, red);
    if (warp % WPR == 0 && (threadIdx.x & 31) == 0) {
#pragma unroll
        for (int r = 0; r < R; ++r)
            if (g * R + r < rows) y[g * R + r] = acc[r];
    }
}

template <class T, int WPR>
__global__ void __launch_bounds__(GV_WARPS * 32) mingru_step_kernel(const T *__restrict__ w, uint32_t wp, uint32_t ld, const T *x,
                                                                    const float *__restrict__ zb, const float *__restrict__ xb, float *state, T *out) {
    __shared__ float red[GV_WARPS][3];
    pdl_trigger();
    const int warp = threadIdx.x >> 5;
    const uint32_t g = blockIdx.x * (GV_WARPS / WPR) + warp / WPR, gi = min(g, wp - 1);
    RowDot<T, 3, 4> d;
#pragma unroll
    for (int r = 0; r < 3; ++r) d.w[r] = w + (size_t)(gi + r * wp) * ld;
    d.start(ld, warp % WPR, WPR);
    d.fetch();
    pdl_wait();
    float acc[3] = {};
    d.run(x, acc);
    group_sum<3, WPR>(acc, red);
    if (warp % WPR == 0 && (threadIdx.x & 31) == 0 && g < wp) {
        float z, cand;
        mingru_gates(acc[0], acc[1], zb[g], xb[g], z, cand);
        const float s = (1.0f - z) * state[g] + z * cand;
        state[g] = s;
        out[g] = Elem<T>::from(s * silu_f32(acc[2]));
    }
}

// Rows [0, ff_p) gate, [ff_p, 2 ff_p) up of w; out = unit(gate, up).
template <class T, int WPR>
__global__ void __launch_bounds__(GV_WARPS * 32) gated_unit_step_kernel(const T *__restrict__ w, uint32_t ff_p, uint32_t ld, const T *x, ExpertAct a, T *out) {
    __shared__ float red[GV_WARPS][2];
    pdl_trigger();
    const int warp = threadIdx.x >> 5;
    const uint32_t g = blockIdx.x * (GV_WARPS / WPR) + warp / WPR, gi = min(g, ff_p - 1);
    RowDot<T, 2, 4> d;
    d.w[0] = w + (size_t)gi * ld;
    d.w[1] = d.w[0] + (size_t)ff_p * ld;
    d.start(ld, warp % WPR, WPR);
    d.fetch();
    pdl_wait();
    float acc[2] = {};
    d.run(x, acc);
    group_sum<2, WPR>(acc, red);
    if (warp % WPR == 0 && (threadIdx.x & 31) == 0 && g < ff_p) out[g] = Elem<T>::from(gated_unit(acc[0], acc[1], a));
}

// grid (row groups, picks).  Every CTA repeats the pick from the router logits; CTA 0 of a pick leaves it for the down step.
template <class T, int WPR>
__global__ void __launch_bounds__(GV_WARPS * 32) expert_gate_up_kernel(const T *__restrict__ w, uint32_t ff_p, uint32_t ld, const T *x,
                                                                       const float *logits, RouterRule rule, ExpertAct a, uint32_t *ids,
                                                                       float *weights, T *act) {
    __shared__ float red[GV_WARPS][2];
    __shared__ float probs[MOE_MAX_EXPERTS];
    __shared__ uint32_t picked[MOE_MAX_USED];
    __shared__ float wt[MOE_MAX_USED];
    pdl_trigger();
    pdl_wait();
    for (uint32_t e = threadIdx.x; e < rule.n_expert; e += blockDim.x) probs[e] = logits[e];
    __syncthreads();
    moe_scores(probs, rule.n_expert, rule.softmax);
    const int warp = threadIdx.x >> 5;
    if (warp == 0) moe_pick(probs, nullptr, rule.n_expert, rule.n_used, rule.renorm, picked, wt);
    __syncthreads();
    const uint32_t s = blockIdx.y, e = picked[s];
    if (blockIdx.x == 0 && threadIdx.x == 0) {
        ids[s] = e;
        weights[s] = wt[s];
    }
    const uint32_t g = blockIdx.x * (GV_WARPS / WPR) + warp / WPR, gi = min(g, ff_p - 1);
    RowDot<T, 2, 4> d;
    d.w[0] = w + ((size_t)e * 2 * ff_p + gi) * ld;
    d.w[1] = d.w[0] + (size_t)ff_p * ld;
    d.start(ld, warp % WPR, WPR);
    d.fetch();
    float acc[2] = {};
    d.run(x, acc);
    group_sum<2, WPR>(acc, red);
    if (warp % WPR == 0 && (threadIdx.x & 31) == 0 && g < ff_p) {
        const float sc = rule.weight_input ? wt[s] : 1.0f;
        act[(size_t)s * ff_p + g] = Elem<T>::from(gated_unit(sc * acc[0], sc * acc[1], a));
    }
}

template <class T, int WPR>
__global__ void __launch_bounds__(GV_WARPS * 32) expert_down_kernel(const T *__restrict__ w, uint32_t rows, uint32_t ld, const T *act, uint32_t n_used,
                                                                    int weight_input, const uint32_t *ids, const float *weights, float *y) {
    __shared__ float red[GV_WARPS][1];
    pdl_trigger();
    pdl_wait();
    const int warp = threadIdx.x >> 5;
    const uint32_t g = blockIdx.x * (GV_WARPS / WPR) + warp / WPR, gi = min(g, rows - 1);
    // the picks' rows are walked as one row of n_used * ld elements, U vectors of it in flight per lane
    constexpr int U = 8;
    const uint32_t nv = ld / Elem<T>::N, all = n_used * nv, step = 32u * WPR;
    float total[1] = {0.0f};
    for (uint32_t c = (warp % WPR) * 32u + (threadIdx.x & 31); c < all; c += U * step) {
        uint4 wb[U], xb[U];
        float sc[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const uint32_t v = c + u * step, s = v / nv;
            if (v < all) {
                wb[u] = ld_stream(reinterpret_cast<const uint4 *>(w + ((size_t)ids[s] * rows + gi) * ld) + (v - s * nv));
                xb[u] = *(reinterpret_cast<const uint4 *>(act) + v);
                sc[u] = weight_input ? 1.0f : weights[s];
            }
        }
#pragma unroll
        for (int u = 0; u < U; ++u)
            if (c + u * step < all) {
                float wf[Elem<T>::N], xf[Elem<T>::N], a = 0.0f;
                Elem<T>::unpack(wb[u], wf);
                Elem<T>::unpack(xb[u], xf);
#pragma unroll
                for (int i = 0; i < Elem<T>::N; ++i) a = fmaf(wf[i], xf[i], a);
                total[0] = fmaf(sc[u], a, total[0]);
            }
    }
    group_sum<1, WPR>(total, red);
    if (warp % WPR == 0 && (threadIdx.x & 31) == 0 && g < rows) y[g] = total[0];
}

}  // namespace

int32_t launch_dense_gemv(const DenseView &w, const void *x, float *y, cudaStream_t st) {
    const bool two = w.rows >= (uint32_t)sm_count() * 28;
    const size_t groups = two ? (w.rows + 1) / 2 : w.rows;
    const int wpr = pick_wpr(groups, (size_t)w.ld * (w.f32 ? 4 : 2), two ? 4 : 8);
    count_launch();
    return with_type(w.f32, [&](auto t) {
        using T = decltype(t);
        return with_wpr(wpr, [&](auto n) {
            constexpr int W = decltype(n)::value;
            return check_cuda(two ? launch_k(gemv_kernel<T, 2, W>, gv_grid(groups, wpr), dim3(GV_WARPS * 32), 0, st, (const T *)w.w, w.rows, w.ld, (const T *)x, y)
                                  : launch_k(gemv_kernel<T, 1, W>, gv_grid(groups, wpr), dim3(GV_WARPS * 32), 0, st, (const T *)w.w, w.rows, w.ld, (const T *)x, y),
                              "dense gemv launch");
        });
    });
}

int32_t launch_mingru_step(const DenseView &w, const void *x, const float *z_bias, const float *x_bias, float *state, void *out, cudaStream_t st) {
    const uint32_t wp = w.rows / 3;
    const int wpr = pick_wpr(wp, (size_t)w.ld * (w.f32 ? 4 : 2), 4);
    count_launch();
    return with_type(w.f32, [&](auto t) {
        using T = decltype(t);
        return with_wpr(wpr, [&](auto n) {
            return check_cuda(launch_k(mingru_step_kernel<T, decltype(n)::value>, gv_grid(wp, wpr), dim3(GV_WARPS * 32), 0, st, (const T *)w.w, wp, w.ld,
                                       (const T *)x, z_bias, x_bias, state, (T *)out),
                              "mingru step launch");
        });
    });
}

int32_t launch_gated_unit_step(const DenseView &w, const void *x, const ExpertAct &a, void *out, cudaStream_t st) {
    const uint32_t ff_p = w.rows / 2;
    const int wpr = pick_wpr(ff_p, (size_t)w.ld * (w.f32 ? 4 : 2), 4);
    count_launch();
    return with_type(w.f32, [&](auto t) {
        using T = decltype(t);
        return with_wpr(wpr, [&](auto n) {
            return check_cuda(launch_k(gated_unit_step_kernel<T, decltype(n)::value>, gv_grid(ff_p, wpr), dim3(GV_WARPS * 32), 0, st, (const T *)w.w, ff_p,
                                       w.ld, (const T *)x, a, (T *)out),
                              "gated unit launch");
        });
    });
}

int32_t launch_expert_gate_up_step(const DenseView &w, const void *x, const float *router_logits, const RouterRule &r, uint32_t ff_p, const ExpertAct &a,
                                   uint32_t *ids, float *weights, void *act, cudaStream_t st) {
    const int wpr = pick_wpr((size_t)ff_p * r.n_used, (size_t)w.ld * (w.f32 ? 4 : 2), 4);
    count_launch();
    return with_type(w.f32, [&](auto t) {
        using T = decltype(t);
        return with_wpr(wpr, [&](auto n) {
            return check_cuda(launch_k(expert_gate_up_kernel<T, decltype(n)::value>, gv_grid(ff_p, wpr, r.n_used), dim3(GV_WARPS * 32), 0, st,
                                       (const T *)w.w, ff_p, w.ld, (const T *)x, router_logits, r, a, ids, weights, (T *)act),
                              "expert gate/up launch");
        });
    });
}

int32_t launch_expert_down_step(const DenseView &w, uint32_t rows_per_expert, const void *act, const RouterRule &r, const uint32_t *ids,
                                const float *weights, float *y, cudaStream_t st) {
    const int wpr = pick_wpr(rows_per_expert, (size_t)w.ld * (w.f32 ? 4 : 2), 2);
    count_launch();
    return with_type(w.f32, [&](auto t) {
        using T = decltype(t);
        return with_wpr(wpr, [&](auto n) {
            return check_cuda(launch_k(expert_down_kernel<T, decltype(n)::value>, gv_grid(rows_per_expert, wpr), dim3(GV_WARPS * 32), 0, st,
                                       (const T *)w.w, rows_per_expert, w.ld, (const T *)act, r.n_used, r.weight_input, ids, weights, y),
                              "expert down launch");
        });
    });
}

}  // namespace cera
