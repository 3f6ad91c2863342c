// Latent attention: keys and values are up-projections of one normed latent per position, so only the latent and one
// rotated key part per position are cached.  This file: what every path needs (norm, rotation, cache append) and the
// latent-space form, in which W_uk is applied to the query and W_uv to the weighted sum of latents - the decode step,
// short prompt portions, and everything in f32.  Scores, softmax and sums are f32.
#include <cooperative_groups.h>

#include <type_traits>

#include "dense.cuh"
#include "mma.cuh"
#include "tma.cuh"

namespace cg = cooperative_groups;

namespace cera {

namespace {

// grid (tokens, parts): part 0 takes the latent, the rotated key part and the gates, the others a share of q.
template <class T>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const float *in, LatentShape s, uint32_t start_pos, const uint32_t *pos_dev,
                                                             const float *__restrict__ c_norm, float eps, const float *__restrict__ rope, T *cache_c,
                                                             T *cache_r, float *q32, T *qt, float *gate) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const uint32_t j = blockIdx.x, pos = (pos_dev ? *pos_dev : start_pos) + j, t = threadIdx.x;
    const float *row = in + (size_t)j * s.in_p, *c = row + s.off_c(), *kr = row + s.off_r(), *gl = row + s.off_g();
    const float *cs = rope + (size_t)pos * s.rot;  // (cos, sin) of the rot / 2 pairs
    auto turned = [&](const float *v, uint32_t i) {  // element i of the rotated vector
        if (i >= s.rot) return 0.0f;
        const float cv = cs[i & ~1u], sv = cs[i | 1u];
        return i & 1 ? v[i] * cv + v[i - 1] * sv : v[i] * cv - v[i + 1] * sv;
    };
    if (blockIdx.y == 0) {
        float ss = 0.0f;
        for (uint32_t i = t; i < s.rank; i += 256) ss += c[i] * c[i];
        const float r = 1.0f / sqrtf(cta_sum(ss, red) / (float)s.rank + eps);
        for (uint32_t i = t; i < s.rank_p; i += 256) cache_c[(size_t)pos * s.rank_p + i] = Elem<T>::from(c[i] * r * c_norm[i]);
        for (uint32_t i = t; i < s.rot_p; i += 256) cache_r[(size_t)pos * s.rot_p + i] = Elem<T>::from(turned(kr, i));
        for (uint32_t h = t; h < s.heads; h += 256) gate[(size_t)j * s.heads + h] = sigmoid_f32(gl[h]);
        return;
    }
    const uint32_t hd = s.dim_p + s.rot_p, total = s.heads * hd;
#pragma unroll 4
    for (uint32_t i = (blockIdx.y - 1) * 256 + t; i < total; i += (gridDim.y - 1) * 256) {
        const uint32_t d = i % hd;
        const float v = d < s.dim_p ? row[i] : turned(row + (i - d) + s.dim_p, d - s.dim_p);
        if (q32) q32[(size_t)j * total + i] = v;
        if (qt) qt[(size_t)j * total + i] = Elem<T>::from(v);
    }
}

// [W_uk_h^T q_h, rotated part] of every (query, head): f32, or for the tensor cores a bf16 high part and the bf16 of what it
// leaves (16 bits of the query survive; the low parts follow all the high parts).  grid (64-column slabs of rank_p, heads, queries), 256 threads = 16 slices of
// the head's dimensions x 16 groups of four columns; weights are fetched ahead of the wait.
template <class T>
__global__ void __launch_bounds__(256) latent_query_kernel(const float *q32, LatentShape s, const T *__restrict__ uk, float *q_lat) {
    using V = typename std::conditional<sizeof(T) == 2, uint2, uint4>::type;  // four elements
    __shared__ float4 part[16][16];
    constexpr int PRE = 8;
    pdl_trigger();
    const uint32_t h = blockIdx.y, j = blockIdx.z, cg = threadIdx.x & 15, sl = threadIdx.x >> 4, c = blockIdx.x * 64 + cg * 4;
    const uint32_t hd = s.dim_p + s.rot_p, ldo = s.rank_p + s.rot_p;
    const float *q = q32 + ((size_t)j * s.heads + h) * hd;
    const T *w = uk + (size_t)h * s.dim_p * s.rank_p + c;
    V ahead[PRE];
#pragma unroll
    for (int i = 0; i < PRE; ++i)
        if (sl + 16 * i < s.dim_p) ahead[i] = *reinterpret_cast<const V *>(w + (size_t)(sl + 16 * i) * s.rank_p);
    pdl_wait();
    float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    auto add = [&](const V &v, float qv) {
        const T *e = reinterpret_cast<const T *>(&v);
        acc.x = fmaf(qv, Elem<T>::to(e[0]), acc.x);
        acc.y = fmaf(qv, Elem<T>::to(e[1]), acc.y);
        acc.z = fmaf(qv, Elem<T>::to(e[2]), acc.z);
        acc.w = fmaf(qv, Elem<T>::to(e[3]), acc.w);
    };
    float qv[PRE];
#pragma unroll
    for (int i = 0; i < PRE; ++i) qv[i] = sl + 16 * i < s.dim_p ? q[sl + 16 * i] : 0.0f;
#pragma unroll
    for (int i = 0; i < PRE; ++i)
        if (sl + 16 * i < s.dim_p) add(ahead[i], qv[i]);
    for (uint32_t d = sl + 16 * PRE; d < s.dim_p; d += 16) add(*reinterpret_cast<const V *>(w + (size_t)d * s.rank_p), q[d]);
    part[sl][cg] = acc;
    __syncthreads();
    const size_t at = ((size_t)j * s.heads + h) * ldo, low = (size_t)gridDim.z * s.heads * ldo;
    auto put = [&](uint32_t i, float v) {
        if constexpr (sizeof(T) == 4) {
            q_lat[at + i] = v;
        } else {
            bf16 *o = reinterpret_cast<bf16 *>(q_lat);
            const bf16 hi = __float2bfloat16_rn(v);
            o[at + i] = hi;
            o[low + at + i] = __float2bfloat16_rn(v - __bfloat162float(hi));
        }
    };
    if (threadIdx.x < 64) {
        float v = 0.0f;
#pragma unroll
        for (int i = 0; i < 16; ++i) v += reinterpret_cast<const float *>(part[i])[threadIdx.x];
        put(blockIdx.x * 64 + threadIdx.x, v);
    } else if (blockIdx.x == 0) {
        for (uint32_t i = threadIdx.x - 64; i < s.rot_p; i += 192) put(s.rank_p + i, q[s.dim_p + i]);
    }
}

constexpr int LA_WARPS = 4, LA_KEYS = 32;

// The f32 form.  One CTA: (split of the keys, 4 HG heads, query).  Tiles of 32 keys in shared memory; a warp owns HG heads: scores with
// lane = key, online softmax, weighted latents with lane = columns.
template <class T, int HG, int NJ>
__global__ void __launch_bounds__(LA_WARPS * 32) latent_split_kernel(const float *q_lat, LatentShape s, const T *cache_c, const T *cache_r, uint32_t start_pos,
                                                                     const uint32_t *len_dev, uint32_t splits, int stages, float *part) {
    constexpr int VN = Elem<T>::N;
    extern __shared__ __align__(16) uint8_t smem[];
    pdl_trigger();
    const uint32_t ql = s.rank_p + s.rot_p, row_b = ql * sizeof(T) + 16, row_v = ql / VN, c_v = s.rank_p / VN;
    float *qs = reinterpret_cast<float *>(smem);  // [LA_WARPS * HG][ql]
    uint8_t *tile = smem + (size_t)LA_WARPS * HG * ql * 4;
    pdl_wait();
    const uint32_t split = blockIdx.x, h0 = blockIdx.y * LA_WARPS * HG, j = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const uint32_t len = len_dev ? *len_dev : start_pos + j + 1;
    const uint32_t per = ((len + splits - 1) / splits + LA_KEYS - 1) / LA_KEYS * LA_KEYS, k0 = min(split * per, len), k1 = min(k0 + per, len);
    {
        const uint32_t live = min((uint32_t)(LA_WARPS * HG), s.heads - h0) * ql / 4;  // the heads of this CTA are one range
        const float4 *src = reinterpret_cast<const float4 *>(q_lat + ((size_t)j * s.heads + h0) * ql);
        for (uint32_t i = threadIdx.x; i < LA_WARPS * HG * ql / 4; i += LA_WARPS * 32) {
            if (i < live) tma::cp_async16(qs + 4 * i, src + i);
            else *reinterpret_cast<float4 *>(qs + 4 * i) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    }
    auto fetch = [&](uint32_t base, int stage) {  // warp = key, lane = vector
        uint8_t *dst = tile + (size_t)stage * LA_KEYS * row_b;
#pragma unroll 4
        for (uint32_t k = warp; k < LA_KEYS; k += LA_WARPS) {
            const T *cr = cache_c + (size_t)(base + k) * s.rank_p, *rr = cache_r + (size_t)(base + k) * s.rot_p;
            for (uint32_t v = lane; v < row_v; v += 32) {
                if (base + k < k1) tma::cp_async16(dst + (size_t)k * row_b + v * 16, v < c_v ? cr + v * VN : rr + (v - c_v) * VN);
                else *reinterpret_cast<uint4 *>(dst + (size_t)k * row_b + v * 16) = make_uint4(0, 0, 0, 0);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float m[HG], l[HG], o[HG][NJ * VN];
#pragma unroll
    for (int g = 0; g < HG; ++g) {
        m[g] = -INFINITY;
        l[g] = 0.0f;
#pragma unroll
        for (int i = 0; i < NJ * VN; ++i) o[g][i] = 0.0f;
    }
    const float *qw = qs + (size_t)warp * HG * ql;
    int stage = 0;
    if (k0 < k1) fetch(k0, 0);
    for (uint32_t base = k0; base < k1; base += LA_KEYS) {
        const bool more = base + LA_KEYS < k1 && stages == 2;
        if (more) fetch(base + LA_KEYS, stage ^ 1);
        if (more) asm volatile("cp.async.wait_group 1;" ::: "memory");
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const uint8_t *tl = tile + (size_t)stage * LA_KEYS * row_b;
        float sc[HG];
#pragma unroll
        for (int g = 0; g < HG; ++g) sc[g] = 0.0f;
        const uint4 *kv = reinterpret_cast<const uint4 *>(tl + (size_t)lane * row_b);
#pragma unroll 4
        for (uint32_t v = 0; v < row_v; ++v) {
            float kf[VN];
            Elem<T>::unpack(kv[v], kf);
#pragma unroll
            for (int g = 0; g < HG; ++g) {
#pragma unroll
                for (int q4 = 0; q4 < VN / 4; ++q4) {
                    const float4 q = *reinterpret_cast<const float4 *>(qw + (size_t)g * ql + v * VN + q4 * 4);
                    sc[g] = fmaf(q.x, kf[q4 * 4], sc[g]);
                    sc[g] = fmaf(q.y, kf[q4 * 4 + 1], sc[g]);
                    sc[g] = fmaf(q.z, kf[q4 * 4 + 2], sc[g]);
                    sc[g] = fmaf(q.w, kf[q4 * 4 + 3], sc[g]);
                }
            }
        }
#pragma unroll
        for (int g = 0; g < HG; ++g) {
            const float v = base + lane < k1 ? sc[g] * s.scale : -INFINITY;
            const float mn = fmaxf(m[g], warp_max(v));  // (the first key of a tile is always valid: mn is finite)
            const float alpha = expf(m[g] - mn);
            sc[g] = expf(v - mn);
            l[g] = l[g] * alpha + warp_sum(sc[g]);
            m[g] = mn;
#pragma unroll
            for (int i = 0; i < NJ * VN; ++i) o[g][i] *= alpha;
        }
        const uint32_t nk = min((uint32_t)LA_KEYS, k1 - base);
#pragma unroll 2
        for (uint32_t k = 0; k < nk; ++k) {
            float p[HG];
#pragma unroll
            for (int g = 0; g < HG; ++g) p[g] = __shfl_sync(0xffffffffu, sc[g], k);
            const uint4 *cv = reinterpret_cast<const uint4 *>(tl + (size_t)k * row_b);
#pragma unroll
            for (int jj = 0; jj < NJ; ++jj) {
                const uint32_t v = jj * 32 + lane;
                if (v < c_v) {
                    float cf[VN];
                    Elem<T>::unpack(cv[v], cf);
#pragma unroll
                    for (int g = 0; g < HG; ++g)
#pragma unroll
                        for (int i = 0; i < VN; ++i) o[g][jj * VN + i] = fmaf(p[g], cf[i], o[g][jj * VN + i]);
                }
            }
        }
        __syncthreads();
        if (stages == 2) stage ^= 1;
        else if (base + LA_KEYS < k1) fetch(base + LA_KEYS, 0);
    }
#pragma unroll
    for (int g = 0; g < HG; ++g) {
        const uint32_t h = h0 + warp * HG + g;
        if (h >= s.heads) continue;
        float *po = part + (((size_t)j * s.heads + h) * splits + split) * (s.rank_p + 2);
        if (lane == 0) {
            po[0] = m[g];
            po[1] = l[g];
        }
#pragma unroll
        for (int jj = 0; jj < NJ; ++jj)
            if (jj * 32 + lane < c_v) {
#pragma unroll
                for (int i = 0; i < VN; ++i) po[2 + (jj * 32 + lane) * VN + i] = o[g][jj * VN + i];
            }
    }
}

// ---- the bf16 form on mma.sync: 16 heads are one operand tile ------------------------------------------------------------
// One CTA: (split of the keys, 16 heads, query); tiles of 64 keys.  Scores: warp = 16 keys, the query as a high and a low
// bf16 part (two products into one f32 accumulator).  Softmax in f32 over the CTA's tile; the weights enter the second
// product as a high and a low part as well.  Weighted latents: warp = a quarter of the latent's columns, NP pairs of 8.
constexpr int LM_KEYS = 64, LM_HEADS = 16, LM_P_LD = LM_KEYS + 8;

template <int NP>
__global__ void __launch_bounds__(128) latent_split_mma_kernel(const bf16 *q, LatentShape s, const bf16 *cache_c, const bf16 *cache_r, uint32_t start_pos,
                                                              const uint32_t *len_dev, uint32_t splits, int stages, float *part) {
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ float row_max[4][LM_HEADS], row_sum[4][LM_HEADS];
    __shared__ __align__(16) bf16 pw[2][LM_HEADS][LM_P_LD];  // weights of the tile: high, low
    pdl_trigger();
    const uint32_t ql = s.rank_p + s.rot_p, ld = ql + 8, row_v = ql / 8, c_v = s.rank_p / 8;
    bf16 *qs = reinterpret_cast<bf16 *>(smem), *tile = qs + 2 * LM_HEADS * ld;  // qs: [high, low][16][ld]
    const uint32_t split = blockIdx.x, h0 = blockIdx.y * LM_HEADS, j = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    pdl_wait();
    const uint32_t len = len_dev ? *len_dev : start_pos + j + 1;
    const uint32_t per = ((len + splits - 1) / splits + LM_KEYS - 1) / LM_KEYS * LM_KEYS, k0 = min(split * per, len), k1 = min(k0 + per, len);
    const size_t low = (size_t)gridDim.z * s.heads * ql;
    for (uint32_t r = warp; r < 2 * LM_HEADS; r += 4) {
        const uint32_t h = h0 + (r & 15);
        const bf16 *src = q + (r >> 4) * low + ((size_t)j * s.heads + h) * ql;
        for (uint32_t v = lane; v < row_v; v += 32) {
            if (h < s.heads) tma::cp_async16(qs + (size_t)r * ld + v * 8, src + v * 8);
            else *reinterpret_cast<uint4 *>(qs + (size_t)r * ld + v * 8) = make_uint4(0, 0, 0, 0);
        }
    }
    auto fetch = [&](uint32_t base, int stage) {
        bf16 *dst = tile + (size_t)stage * LM_KEYS * ld;
        for (uint32_t k = warp; k < LM_KEYS; k += 4) {
            const bf16 *cr = cache_c + (size_t)(base + k) * s.rank_p, *rr = cache_r + (size_t)(base + k) * s.rot_p;
            for (uint32_t v = lane; v < row_v; v += 32) {
                if (base + k < k1) tma::cp_async16(dst + (size_t)k * ld + v * 8, v < c_v ? cr + v * 8 : rr + (v - c_v) * 8);
                else *reinterpret_cast<uint4 *>(dst + (size_t)k * ld + v * 8) = make_uint4(0, 0, 0, 0);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float o[NP][2][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};  // rows lane / 4 and lane / 4 + 8
#pragma unroll
    for (int i = 0; i < NP; ++i)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[i][n][e] = 0.0f;
    const uint32_t r0 = lane >> 2, col2 = (lane & 3) * 2, cols = s.rank_p / 4, c_base = warp * cols;  // cols: a multiple of 16
    const float sc2 = s.scale * 1.44269504088896340736f;
    int stage = 0;
    if (k0 < k1) fetch(k0, 0);
    for (uint32_t base = k0; base < k1; base += LM_KEYS) {
        const bool more = base + LM_KEYS < k1 && stages == 2;
        if (more) fetch(base + LM_KEYS, stage ^ 1);
        if (more) asm volatile("cp.async.wait_group 1;" ::: "memory");
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const bf16 *tl = tile + (size_t)stage * LM_KEYS * ld;
        float sc[2][4] = {};
        {
            const bf16 *qa = qs + (size_t)(lane & 15) * ld + (lane >> 4) * 8;
            const bf16 *kb = tl + (size_t)(warp * 16 + (lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8;
#pragma unroll 4
            for (uint32_t k = 0; k < ql; k += 16) {
                uint32_t ah[4], al[4], b[4];
                ldsm4(ah, qa + k);
                ldsm4(al, qa + (size_t)LM_HEADS * ld + k);
                ldsm4(b, kb + k);
                mma_bf16(sc[0], ah, b[0], b[1]);
                mma_bf16(sc[1], ah, b[2], b[3]);
                mma_bf16(sc[0], al, b[0], b[1]);
                mma_bf16(sc[1], al, b[2], b[3]);
            }
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t key = base + warp * 16 + n * 8 + col2 + (e & 1);
                sc[n][e] = key < k1 ? sc[n][e] * sc2 : -INFINITY;
                mx[e >> 1] = fmaxf(mx[e >> 1], sc[n][e]);
            }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            if ((lane & 3) == 0) row_max[warp][r0 + 8 * r] = mx[r];
        }
        __syncthreads();
        float alpha[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const uint32_t row = r0 + 8 * r;
            // the first key of a tile is always valid: the maximum is finite
            const float mn = fmaxf(m[r], fmaxf(fmaxf(row_max[0][row], row_max[1][row]), fmaxf(row_max[2][row], row_max[3][row])));
            alpha[r] = exp2f(m[r] - mn);
            m[r] = mn;
            l[r] *= alpha[r];
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const float e0 = exp2f(sc[n][2 * r] - m[r]), e1 = exp2f(sc[n][2 * r + 1] - m[r]);
                l[r] += e0 + e1;
                const __nv_bfloat162 hi = __floats2bfloat162_rn(e0, e1);
                const float2 hf = __bfloat1622float2(hi);
                const uint32_t c = warp * 16 + n * 8 + col2;
                *reinterpret_cast<__nv_bfloat162 *>(&pw[0][r0 + 8 * r][c]) = hi;
                *reinterpret_cast<__nv_bfloat162 *>(&pw[1][r0 + 8 * r][c]) = __floats2bfloat162_rn(e0 - hf.x, e1 - hf.y);
            }
#pragma unroll
        for (int i = 0; i < NP; ++i)
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[i][n][e] *= alpha[e >> 1];
        __syncthreads();
        const bf16 *vb = tl + (size_t)((lane & 7) + ((lane >> 3) & 1) * 8) * ld + c_base + (lane >> 4) * 8;
#pragma unroll 1
        for (uint32_t k = 0; k < LM_KEYS; k += 16) {
            uint32_t ph[4], pl[4];
            ldsm4(ph, &pw[0][lane & 15][k + (lane >> 4) * 8]);
            ldsm4(pl, &pw[1][lane & 15][k + (lane >> 4) * 8]);
#pragma unroll
            for (int i = 0; i < NP; ++i)
                if ((uint32_t)i * 16 < cols) {
                    uint32_t b[4];
                    ldsm4_trans(b, vb + (size_t)k * ld + i * 16);
                    mma_bf16(o[i][0], ph, b[0], b[1]);
                    mma_bf16(o[i][1], ph, b[2], b[3]);
                    mma_bf16(o[i][0], pl, b[0], b[1]);
                    mma_bf16(o[i][1], pl, b[2], b[3]);
                }
        }
        __syncthreads();
        if (stages == 2) stage ^= 1;
        else if (base + LM_KEYS < k1) fetch(base + LM_KEYS, 0);
    }
    // per row: maximum (natural units), sum of weights over the four warps' keys, weighted latents
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        if ((lane & 3) == 0) row_sum[warp][r0 + 8 * r] = l[r];
    }
    asm volatile("cp.async.wait_all;" ::: "memory");  // a split without keys has still asked for its queries
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const uint32_t row = r0 + 8 * r, h = h0 + row;
        if (h >= s.heads) continue;
        float *po = part + (((size_t)j * s.heads + h) * splits + split) * (s.rank_p + 2);
        if (warp == 0 && (lane & 3) == 0) {
            po[0] = m[r] * 0.69314718055994530942f;
            po[1] = row_sum[0][row] + row_sum[1][row] + row_sum[2][row] + row_sum[3][row];
        }
#pragma unroll
        for (int i = 0; i < NP; ++i)
            if ((uint32_t)i * 16 < cols) {
#pragma unroll
                for (int n = 0; n < 2; ++n)
                    *reinterpret_cast<float2 *>(po + 2 + c_base + i * 16 + n * 8 + col2) = make_float2(o[i][n][2 * r], o[i][n][2 * r + 1]);
            }
    }
}

template <int NP>
int32_t launch_split_mma(const LatentScratch &ws, const LatentShape &s, const void *cc, const void *cr, size_t n, size_t start_pos, const uint32_t *len_dev,
                         uint32_t splits, cudaStream_t st) {
    const size_t ld = s.rank_p + s.rot_p + 8, qb = 2 * LM_HEADS * ld * 2, tb = LM_KEYS * ld * 2;
    const int stages = qb + 2 * tb <= 215 * 1024 ? 2 : 1;
    const size_t bytes = qb + stages * tb;
    if (bytes > 215 * 1024) return fail(CERA_CUDA_ERR_UNSUPPORTED, "latent attention: rank %u with %u rotated dimensions", s.rank, s.rot);
    auto k = latent_split_mma_kernel<NP>;
    CERA_CUDA_TRY(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 215 * 1024));
    count_launch();
    return check_cuda(launch_k(k, dim3(splits, (s.heads + LM_HEADS - 1) / LM_HEADS, (unsigned)n), dim3(128), bytes, st, (const bf16 *)ws.q_lat, s, (const bf16 *)cc,
                               (const bf16 *)cr, (uint32_t)start_pos, len_dev, splits, stages, ws.part),
                      "latent split launch");
}

// A cluster of four CTAs per (head, query): each combines the splits for a quarter of the latent's columns - the sink counts
// in the denominator - and hands its quarter to the others through distributed shared memory; each then takes a quarter of
// the head's rows of W_uv.
constexpr uint32_t MERGE_CL = 4;
template <class T>
__global__ void __cluster_dims__(MERGE_CL, 1, 1) __launch_bounds__(256) latent_merge_kernel(const float *part, LatentShape s, uint32_t splits,
                                                                                          const float *__restrict__ sink, const float *gate,
                                                                                          const T *__restrict__ uv, T *out, size_t ldo) {
    extern __shared__ __align__(16) float lat[];  // [rank_p]
    __shared__ float wt[LATENT_MAX_SPLITS];
    __shared__ float2 sums[4][64];
    cg::cluster_group cluster = cg::this_cluster();
    pdl_trigger();
    const uint32_t h = blockIdx.y, j = blockIdx.z, ps = s.rank_p + 2, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, cr = cluster.block_rank();
    const uint32_t slab = (s.vdim_p + MERGE_CL - 1) / MERGE_CL, v0 = cr * slab, v1 = min(v0 + slab, s.vdim_p);
    pdl_wait();
    const float *p = part + ((size_t)j * s.heads + h) * splits * ps;
    if (warp == 0) {
        constexpr int PER = LATENT_MAX_SPLITS / 32;
        const float sk = sink[h];
        float ms[PER], ls[PER], mx = sk;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const uint32_t sp = lane + 32 * i;
            ms[i] = sp < splits ? p[(size_t)sp * ps] : -INFINITY;
            ls[i] = sp < splits ? p[(size_t)sp * ps + 1] : 0.0f;
            mx = fmaxf(mx, ms[i]);
        }
        mx = warp_max(mx);
        float den = 0.0f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            ms[i] = expf(ms[i] - mx);
            den += ms[i] * ls[i];
        }
        den = warp_sum(den) + expf(sk - mx);
#pragma unroll
        for (int i = 0; i < PER; ++i)
            if (lane + 32 * i < splits) wt[lane + 32 * i] = ms[i] / den;
    }
    cluster.sync();  // every CTA of the cluster runs before its shared memory is written from outside
    const uint32_t quarter = s.rank_p / MERGE_CL, sub = threadIdx.x >> 6, tc = threadIdx.x & 63;  // rank_p is a multiple of 64
    for (uint32_t c0 = 0; c0 < quarter; c0 += 128) {  // 64 threads x 2 columns, four of them share the splits
        const uint32_t c = c0 + 2 * tc;
        float2 a = make_float2(0.0f, 0.0f);
        if (c < quarter) {
            const float *src = p + 2 + cr * quarter + c;
#pragma unroll 8
            for (uint32_t i = sub; i < splits; i += 4) {
                const float2 v = *reinterpret_cast<const float2 *>(src + (size_t)i * ps);
                a.x = fmaf(wt[i], v.x, a.x);
                a.y = fmaf(wt[i], v.y, a.y);
            }
        }
        sums[sub][tc] = a;
        __syncthreads();
        if (sub == 0 && c < quarter) {
#pragma unroll
            for (int i = 1; i < 4; ++i) {
                a.x += sums[i][tc].x;
                a.y += sums[i][tc].y;
            }
            sums[0][tc] = a;
        }
        __syncthreads();
        // thread group `sub` writes the pair into CTA `sub` of the cluster
        if (c < quarter) *reinterpret_cast<float2 *>(cluster.map_shared_rank(lat, sub) + cr * quarter + c) = sums[0][tc];
        __syncthreads();
    }
    cluster.sync();
    const float gt = gate[(size_t)j * s.heads + h];
#pragma unroll 4
    for (uint32_t v = v0 + warp; v < v1; v += 8) {
        const uint4 *w = reinterpret_cast<const uint4 *>(uv + ((size_t)h * s.vdim_p + v) * s.rank_p);
        float acc = 0.0f;
        for (uint32_t c = lane; c < s.rank_p / Elem<T>::N; c += 32) {
            float wf[Elem<T>::N];
            Elem<T>::unpack(__ldg(w + c), wf);
#pragma unroll
            for (int i = 0; i < Elem<T>::N; ++i) acc = fmaf(wf[i], lat[c * Elem<T>::N + i], acc);
        }
        acc = warp_sum(acc);
        if (lane == 0) out[j * ldo + (size_t)h * s.vdim_p + v] = Elem<T>::from(acc * gt);
    }
}

template <class T, int HG, int NJ>
int32_t launch_split(const LatentScratch &ws, const LatentShape &s, const void *cc, const void *cr, size_t n, size_t start_pos, const uint32_t *len_dev,
                     uint32_t splits, cudaStream_t st) {
    const uint32_t ql = s.rank_p + s.rot_p;
    const size_t qb = (size_t)LA_WARPS * HG * ql * 4, tb = (size_t)LA_KEYS * (ql * sizeof(T) + 16);
    const int stages = qb + 2 * tb <= 220 * 1024 ? 2 : 1;
    const size_t smem = qb + stages * tb;
    if (smem > 220 * 1024) return fail(CERA_CUDA_ERR_UNSUPPORTED, "latent attention: rank %u with %u rotated dimensions", s.rank, s.rot);
    auto k = latent_split_kernel<T, HG, NJ>;
    CERA_CUDA_TRY(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    count_launch();
    return check_cuda(launch_k(k, dim3(splits, (s.heads + LA_WARPS * HG - 1) / (LA_WARPS * HG), (unsigned)n), dim3(LA_WARPS * 32), smem, st, (const float *)ws.q_lat,
                               s, (const T *)cc, (const T *)cr, (uint32_t)start_pos, len_dev, splits, stages, ws.part),
                      "latent split launch");
}

template <class T>
int32_t latent_attention(const float *q32, const LatentShape &s, const void *uk, const void *uv, const void *cc, const void *cr, const float *sink,
                         const float *gate, size_t n, size_t start_pos, const uint32_t *len_dev, uint32_t splits, const LatentScratch &ws, void *out,
                         size_t ldo, cudaStream_t st) {
    count_launch();
    CERA_CUDA_TRY(launch_k(latent_query_kernel<T>, dim3(s.rank_p / 64, s.heads, (unsigned)n), dim3(256), 0, st, q32, s, (const T *)uk, ws.q_lat));
    int32_t rc;
    if constexpr (sizeof(T) == 2) {
        rc = s.rank_p <= 256   ? launch_split_mma<4>(ws, s, cc, cr, n, start_pos, len_dev, splits, st)
             : s.rank_p <= 512 ? launch_split_mma<8>(ws, s, cc, cr, n, start_pos, len_dev, splits, st)
                               : launch_split_mma<16>(ws, s, cc, cr, n, start_pos, len_dev, splits, st);
    } else {
        const uint32_t nj = (s.rank_p / 4 + 31) / 32;
        auto split = [&](auto hg) -> int32_t {
            constexpr int HG = decltype(hg)::value;
            if (nj <= 1) return launch_split<T, HG, 1>(ws, s, cc, cr, n, start_pos, len_dev, splits, st);
            if (nj <= 2) return launch_split<T, HG, 2>(ws, s, cc, cr, n, start_pos, len_dev, splits, st);
            if (nj <= 4) return launch_split<T, HG, 4>(ws, s, cc, cr, n, start_pos, len_dev, splits, st);
            return launch_split<T, HG, 8>(ws, s, cc, cr, n, start_pos, len_dev, splits, st);
        };
        rc = s.heads <= 8 ? split(std::integral_constant<int, 1>{}) : split(std::integral_constant<int, 4>{});  // few heads: one per warp
    }
    CERA_TRY(rc);
    count_launch();
    return check_cuda(launch_k(latent_merge_kernel<T>, dim3(MERGE_CL, s.heads, (unsigned)n), dim3(256), (size_t)s.rank_p * 4, st, (const float *)ws.part, s, splits,
                               sink, gate, (const T *)uv, (T *)out, ldo),
                      "latent merge launch");
}

}  // namespace

int32_t launch_latent_prepare(const float *in, const LatentShape &s, size_t n, size_t start_pos, const uint32_t *pos_dev, const float *c_norm, float eps,
                              const float *rope_table, void *cache_c, void *cache_r, int f32, float *q32, void *qt, float *gate, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    const uint32_t total = s.q_ld(), per = n == 1 ? 512 : 2048;  // q elements of a CTA
    const dim3 grid((unsigned)n, 1 + (total + per - 1) / per);
    count_launch();
    if (f32)
        return check_cuda(launch_k(latent_prepare_kernel<float>, grid, dim3(256), 0, st, in, s, (uint32_t)start_pos, pos_dev, c_norm, eps,
                                   rope_table, (float *)cache_c, (float *)cache_r, q32, (float *)qt, gate), "latent prepare launch");
    return check_cuda(launch_k(latent_prepare_kernel<bf16>, grid, dim3(256), 0, st, in, s, (uint32_t)start_pos, pos_dev, c_norm, eps, rope_table,
                               (bf16 *)cache_c, (bf16 *)cache_r, q32, (bf16 *)qt, gate), "latent prepare launch");
}

int32_t launch_latent_attention(const float *q32, const LatentShape &s, const DenseView &uk, const DenseView &uv, const void *cache_c, const void *cache_r,
                                const float *sink, const float *gate, size_t n, size_t start_pos, const uint32_t *len_dev, uint32_t splits,
                                const LatentScratch &ws, void *out, size_t ldo, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    if (splits == 0 || splits > LATENT_MAX_SPLITS || n * splits > LATENT_MAX_SPLITS)
        return fail(CERA_CUDA_ERR_BAD_ARG, "latent attention: %zu queries x %u splits", n, splits);
    return uk.f32 ? latent_attention<float>(q32, s, uk.w, uv.w, cache_c, cache_r, sink, gate, n, start_pos, len_dev, splits, ws, out, ldo, st)
                  : latent_attention<bf16>(q32, s, uk.w, uv.w, cache_c, cache_r, sink, gate, n, start_pos, len_dev, splits, ws, out, ldo, st);
}

}  // namespace cera
