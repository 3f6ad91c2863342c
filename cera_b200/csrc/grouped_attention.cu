// Attention whose query heads share key / value heads in groups: bias, rotation and unit-root-mean-square norm of queries
// and keys, cache append, and attention over the cache for one query or a few (decode, short portions, everything in f32).
// Long bf16 portions take attention_tc.cu.  Keys are cached by position, values transposed, which is what the products of
// both paths want.  Scores, softmax and sums are f32.
#include "dense.cuh"
#include "tma.cuh"

namespace cera {

namespace {

constexpr int GP_WARPS = 8;

// One warp per head of q and of k; with one token also a warp per 64 values.  grid (tokens, parts).
template <class T>
__global__ void __launch_bounds__(GP_WARPS * 32) grouped_prepare_kernel(const float *in, GroupedShape s, uint32_t start_pos, const uint32_t *pos_dev,
                                                                        const float *__restrict__ bias, const float *__restrict__ rope, T *cache_k, T *cache_v,
                                                                        size_t ld_v, float *q32, T *qt) {
    pdl_trigger();
    pdl_wait();
    const uint32_t j = blockIdx.x, pos = (pos_dev ? *pos_dev : start_pos) + j, lane = threadIdx.x & 31, v = blockIdx.y * GP_WARPS + (threadIdx.x >> 5);
    const float *row = in + (size_t)j * s.in_p;
    if (v >= s.heads + s.kv_heads) {
        if (gridDim.x > 1) return;  // a portion's values: values_append_kernel
        const uint32_t first = (v - s.heads - s.kv_heads) * 64, n_v = s.kv_heads * s.vdim_p;
        for (uint32_t i = first + lane; i < min(first + 64, n_v); i += 32)
            cache_v[(size_t)i * ld_v + pos] = Elem<T>::from(row[s.off_v() + i] + bias[s.off_v() + i]);
        return;
    }
    const float2 *x = reinterpret_cast<const float2 *>(row + v * s.dim_p), *b = reinterpret_cast<const float2 *>(bias + v * s.dim_p);
    const float2 *cs = reinterpret_cast<const float2 *>(rope + (size_t)pos * s.rot);  // (cos, sin) of the rot / 2 pairs
    auto turned = [&](uint32_t i) {  // pair i
        float2 a = x[i];
        const float2 c = b[i];
        a.x += c.x;
        a.y += c.y;
        if (2 * i < s.rot) {
            const float2 t = cs[i];
            a = make_float2(a.x * t.x - a.y * t.y, a.y * t.x + a.x * t.y);
        }
        return a;
    };
    constexpr int KEEP = 4;  // pairs a lane holds in registers
    float2 keep[KEEP];
    float ss = 0.0f;
    const uint32_t pairs = s.dim_p / 2;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        keep[k] = lane + 32 * k < pairs ? turned(lane + 32 * k) : make_float2(0.0f, 0.0f);
        ss += keep[k].x * keep[k].x + keep[k].y * keep[k].y;
    }
    for (uint32_t i = lane + 32 * KEEP; i < pairs; i += 32) {
        const float2 a = turned(i);
        ss += a.x * a.x + a.y * a.y;
    }
    const float r = s.qk_norm ? 1.0f / sqrtf(warp_sum(ss) / (float)s.dim + s.eps) : 1.0f;
    const bool is_k = v >= s.heads;
    T *kt = cache_k + (size_t)pos * s.kv_heads * s.dim_p + (size_t)(is_k ? v - s.heads : 0) * s.dim_p;
    const size_t qo = (size_t)j * s.q_ld() + (size_t)v * s.dim_p;
    auto put = [&](uint32_t i, float2 a) {
        a.x *= r;
        a.y *= r;
        if (is_k) {
            kt[2 * i] = Elem<T>::from(a.x);
            kt[2 * i + 1] = Elem<T>::from(a.y);
            return;
        }
        if (q32) *reinterpret_cast<float2 *>(q32 + qo + 2 * i) = a;
        if (qt) {
            qt[qo + 2 * i] = Elem<T>::from(a.x);
            qt[qo + 2 * i + 1] = Elem<T>::from(a.y);
        }
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
        if (lane + 32 * k < pairs) put(lane + 32 * k, keep[k]);
    for (uint32_t i = lane + 32 * KEEP; i < pairs; i += 32) put(i, turned(i));
}

// Values of a portion into the transposed cache: 32 tokens x 32 values through shared memory.
template <class T>
__global__ void __launch_bounds__(256) values_append_kernel(const float *in, size_t in_p, uint32_t off, const float *__restrict__ bias, uint32_t n, uint32_t rows,
                                                            uint32_t start_pos, T *cache_v, size_t ld_v) {
    __shared__ float tile[32][33];
    pdl_trigger();
    pdl_wait();
    const uint32_t t0 = blockIdx.x * 32, r0 = blockIdx.y * 32, a = threadIdx.x & 31, b = threadIdx.x >> 5;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const uint32_t t = t0 + b + 8 * i;
        if (t < n && r0 + a < rows) tile[b + 8 * i][a] = in[(size_t)t * in_p + off + r0 + a] + bias[off + r0 + a];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const uint32_t r = r0 + b + 8 * i;
        if (r < rows && t0 + a < n) cache_v[(size_t)r * ld_v + start_pos + t0 + a] = Elem<T>::from(tile[a][b + 8 * i]);
    }
}

constexpr int GS_WARPS = 8;

// One CTA: (split of the keys, up to `hc` heads of one group, query).  Tiles of `tk` keys in shared memory: scores with
// lane = key, online softmax with warp = head, weighted values with lane = value; NI (head, 32 values) items a warp.
template <class T, int NI>
__global__ void __launch_bounds__(GS_WARPS * 32) grouped_split_kernel(const float *q32, GroupedShape s, const T *cache_k, const T *cache_v, size_t ld_v,
                                                                      uint32_t start_pos, const uint32_t *len_dev, uint32_t splits, uint32_t hc, uint32_t tk,
                                                                      float *part) {
    constexpr int VN = Elem<T>::N;
    extern __shared__ __align__(16) uint8_t smem[];
    pdl_trigger();
    const uint32_t krow = s.dim_p * sizeof(T) + 16, vrow = tk * sizeof(T) + 16, kv = s.dim_p / VN, vv = tk / VN;
    uint8_t *kt = smem, *vt = kt + (size_t)tk * krow;
    float *qs = reinterpret_cast<float *>(vt + (size_t)s.vdim_p * vrow), *sc = qs + hc * s.dim_p, *stat = sc + hc * tk;  // stat: m, l, alpha of hc heads
    const uint32_t ratio = s.heads / s.kv_heads, chunks = (ratio + hc - 1) / hc, g = blockIdx.y / chunks, i0 = blockIdx.y % chunks * hc, nh = min(hc, ratio - i0),
                   h0 = g * ratio + i0, j = blockIdx.z, split = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    pdl_wait();
    const uint32_t len = len_dev ? *len_dev : start_pos + j + 1;
    const uint32_t per = ((len + splits - 1) / splits + 63) / 64 * 64, k0 = min(split * per, len), k1 = min(k0 + per, len);
    for (uint32_t i = threadIdx.x; i < nh * s.dim_p / 4; i += GS_WARPS * 32)
        tma::cp_async16(qs + 4 * i, q32 + (size_t)j * s.q_ld() + (size_t)h0 * s.dim_p + 4 * i);
    for (uint32_t i = threadIdx.x; i < hc; i += GS_WARPS * 32) {
        stat[i] = -INFINITY;
        stat[hc + i] = 0.0f;
    }
    const uint32_t dchunks = (s.vdim_p + 31) / 32, items = nh * dchunks;
    float o[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) o[i] = 0.0f;
    for (uint32_t base = k0; base < k1; base += tk) {
        for (uint32_t i = threadIdx.x; i < tk * kv; i += GS_WARPS * 32) {
            const uint32_t k = i / kv, c = i - k * kv;
            uint8_t *dst = kt + (size_t)k * krow + c * 16;
            if (base + k < k1) tma::cp_async16(dst, cache_k + ((size_t)(base + k) * s.kv_heads + g) * s.dim_p + c * VN);
            else *reinterpret_cast<uint4 *>(dst) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        for (uint32_t i = threadIdx.x; i < s.vdim_p * vv; i += GS_WARPS * 32) {  // columns past the end meet zero weights
            const uint32_t d = i / vv, c = i - d * vv;
            tma::cp_async16(vt + (size_t)d * vrow + c * 16, cache_v + ((size_t)g * s.vdim_p + d) * ld_v + base + c * VN);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const uint32_t kgroups = (tk + 31) / 32;
        for (uint32_t it = warp; it < nh * kgroups; it += GS_WARPS) {
            const uint32_t hh = it / kgroups, k = (it - hh * kgroups) * 32 + lane;
            if (k >= tk) continue;
            const float *q = qs + hh * s.dim_p;
            const uint4 *kr = reinterpret_cast<const uint4 *>(kt + (size_t)k * krow);
            float acc = 0.0f;
#pragma unroll 4
            for (uint32_t c = 0; c < kv; ++c) {
                float kf[VN];
                Elem<T>::unpack(kr[c], kf);
#pragma unroll
                for (int e = 0; e < VN; ++e) acc = fmaf(q[c * VN + e], kf[e], acc);
            }
            acc *= s.scale;
            if (s.softcap > 0.0f) acc = s.softcap * tanhf(acc / s.softcap);
            sc[hh * tk + k] = base + k < k1 ? acc : -INFINITY;
        }
        __syncthreads();
        for (uint32_t hh = warp; hh < nh; hh += GS_WARPS) {
            float mx = -INFINITY;
            for (uint32_t k = lane; k < tk; k += 32) mx = fmaxf(mx, sc[hh * tk + k]);
            const float old = stat[hh], mn = fmaxf(old, warp_max(mx));  // the first key of a tile is valid: finite
            float sum = 0.0f;
            for (uint32_t k = lane; k < tk; k += 32) {
                const float e = expf(sc[hh * tk + k] - mn);
                sc[hh * tk + k] = e;
                sum += e;
            }
            sum = warp_sum(sum);
            __syncwarp();
            if (lane == 0) {
                const float alpha = expf(old - mn);
                stat[hh] = mn;
                stat[hc + hh] = stat[hc + hh] * alpha + sum;
                stat[2 * hc + hh] = alpha;
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const uint32_t it = warp + i * GS_WARPS;
            if (it >= items) continue;
            const uint32_t hh = it / dchunks, d = (it - hh * dchunks) * 32 + lane;
            if (d >= s.vdim_p) continue;
            const uint4 *vr = reinterpret_cast<const uint4 *>(vt + (size_t)d * vrow);
            const float *w = sc + hh * tk;
            float acc = o[i] * stat[2 * hc + hh];
#pragma unroll 4
            for (uint32_t c = 0; c < vv; ++c) {
                float vf[VN];
                Elem<T>::unpack(vr[c], vf);
#pragma unroll
                for (int e = 0; e < VN; ++e) acc = fmaf(w[c * VN + e], vf[e], acc);
            }
            o[i] = acc;
        }
        __syncthreads();
    }
    asm volatile("cp.async.wait_all;" ::: "memory");  // a split without keys has still asked for its queries
    __syncthreads();
    const size_t ps = s.vdim_p + 2;
    float *po = part + (((size_t)j * s.heads + h0) * splits + split) * ps;
    for (uint32_t hh = threadIdx.x; hh < nh; hh += GS_WARPS * 32) {
        po[(size_t)hh * splits * ps] = stat[hh];
        po[(size_t)hh * splits * ps + 1] = stat[hc + hh];
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const uint32_t it = warp + i * GS_WARPS;
        if (it >= items) continue;
        const uint32_t hh = it / dchunks, d = (it - hh * dchunks) * 32 + lane;
        if (d < s.vdim_p) po[(size_t)hh * splits * ps + 2 + d] = o[i];
    }
}

// grid (heads, queries): the splits' sums under a common maximum.
template <class T>
__global__ void __launch_bounds__(256) grouped_merge_kernel(const float *part, GroupedShape s, uint32_t splits, T *out, size_t ldo) {
    __shared__ float wt[KV_MAX_SPLITS];
    __shared__ float2 sums[8][32];
    pdl_trigger();
    pdl_wait();
    const uint32_t h = blockIdx.x, j = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const size_t ps = s.vdim_p + 2;
    const float *p = part + ((size_t)j * s.heads + h) * splits * ps;
    if (threadIdx.x < 32) {
        constexpr int PER = KV_MAX_SPLITS / 32;
        float ms[PER], ls[PER], mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const uint32_t sp = lane + 32 * i;
            ms[i] = sp < splits ? p[sp * ps] : -INFINITY;
            ls[i] = sp < splits ? p[sp * ps + 1] : 0.0f;
            mx = fmaxf(mx, ms[i]);
        }
        mx = warp_max(mx);  // finite: the query sees itself
        float den = 0.0f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            ms[i] = expf(ms[i] - mx);
            den += ms[i] * ls[i];
        }
        den = warp_sum(den);
#pragma unroll
        for (int i = 0; i < PER; ++i)
            if (lane + 32 * i < splits) wt[lane + 32 * i] = ms[i] / den;
    }
    __syncthreads();
    for (uint32_t d0 = 0; d0 < s.vdim_p; d0 += 64) {  // a lane two values, a warp every eighth split
        const uint32_t d = d0 + 2 * lane;
        float2 acc = make_float2(0.0f, 0.0f);
        if (d < s.vdim_p) {
#pragma unroll 8
            for (uint32_t i = warp; i < splits; i += 8) {
                const float2 v = *reinterpret_cast<const float2 *>(p + i * ps + 2 + d);
                acc.x = fmaf(wt[i], v.x, acc.x);
                acc.y = fmaf(wt[i], v.y, acc.y);
            }
        }
        sums[warp][lane] = acc;
        __syncthreads();
        if (warp == 0 && d < s.vdim_p) {
#pragma unroll
            for (int i = 1; i < 8; ++i) {
                acc.x += sums[i][lane].x;
                acc.y += sums[i][lane].y;
            }
            T *o = out + j * ldo + (size_t)h * s.vdim_p + d;
            o[0] = Elem<T>::from(acc.x);
            o[1] = Elem<T>::from(acc.y);
        }
        __syncthreads();
    }
}

template <class T>
int32_t grouped_attention(const float *q32, const GroupedShape &s, const void *ck, const void *cv, size_t ld_v, size_t n, size_t start_pos,
                          const uint32_t *len_dev, uint32_t splits, float *part, void *out, size_t ldo, cudaStream_t st) {
    constexpr uint32_t MOST = 8;  // items a warp accumulates
    const uint32_t ratio = s.heads / s.kv_heads, dchunks = (s.vdim_p + 31) / 32;
    uint32_t hc = ratio < 16 ? ratio : 16;
    while (hc > 1 && hc * dchunks > GS_WARPS * MOST) hc = (hc + 1) / 2;
    const uint32_t items = hc * dchunks, ni = (items + GS_WARPS - 1) / GS_WARPS;
    auto bytes = [&](uint32_t tk) {
        return (size_t)tk * (s.dim_p * sizeof(T) + 16) + (size_t)s.vdim_p * (tk * sizeof(T) + 16) + ((size_t)hc * (s.dim_p + tk + 3)) * 4;
    };
    uint32_t tk = 64;
    while (tk > 8 && bytes(tk) > 220 * 1024) tk /= 2;
    if (ni > MOST || bytes(tk) > 220 * 1024) return fail(CERA_CUDA_ERR_UNSUPPORTED, "attention: heads of %u / %u", s.dim, s.vdim);
    const dim3 grid(splits, s.kv_heads * ((ratio + hc - 1) / hc), (unsigned)n);
    auto go = [&](auto k) {
        CERA_CUDA_TRY(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        count_launch();
        return check_cuda(launch_k(k, grid, dim3(GS_WARPS * 32), bytes(tk), st, q32, s, (const T *)ck, (const T *)cv, ld_v, (uint32_t)start_pos, len_dev, splits,
                                   hc, tk, part),
                          "attention split launch");
    };
    CERA_TRY(ni <= 1 ? go(grouped_split_kernel<T, 1>) : ni <= 2 ? go(grouped_split_kernel<T, 2>) : ni <= 4 ? go(grouped_split_kernel<T, 4>) : go(grouped_split_kernel<T, 8>));
    count_launch();
    return check_cuda(launch_k(grouped_merge_kernel<T>, dim3(s.heads, (unsigned)n), dim3(256), 0, st, (const float *)part, s, splits, (T *)out, ldo), "attention merge launch");
}

}  // namespace

int32_t launch_grouped_prepare(const float *in, const GroupedShape &s, size_t n, size_t start_pos, const uint32_t *pos_dev, const float *bias,
                               const float *rope_table, void *cache_k, void *cache_v, size_t ld_v, int f32, float *q32, void *qt, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    const uint32_t n_v = s.kv_heads * s.vdim_p, vectors = s.heads + s.kv_heads + (n == 1 ? (n_v + 63) / 64 : 0);
    const dim3 grid((unsigned)n, (vectors + GP_WARPS - 1) / GP_WARPS), vgrid((unsigned)((n + 31) / 32), (n_v + 31) / 32);
    auto typed = [&](auto t) {
        using T = decltype(t);
        count_launch();
        CERA_CUDA_TRY(launch_k(grouped_prepare_kernel<T>, grid, dim3(GP_WARPS * 32), 0, st, in, s, (uint32_t)start_pos, pos_dev, bias, rope_table, (T *)cache_k,
                               (T *)cache_v, ld_v, q32, (T *)qt));
        if (n == 1) return (int32_t)CERA_CUDA_OK;
        count_launch();
        return check_cuda(launch_k(values_append_kernel<T>, vgrid, dim3(256), 0, st, in, (size_t)s.in_p, s.off_v(), bias, (uint32_t)n, n_v, (uint32_t)start_pos,
                                   (T *)cache_v, ld_v),
                          "values append launch");
    };
    return f32 ? typed(float{}) : typed(bf16{});
}

int32_t launch_grouped_attention(const float *q32, const GroupedShape &s, const void *cache_k, const void *cache_v, size_t ld_v, int f32, size_t n,
                                 size_t start_pos, const uint32_t *len_dev, uint32_t splits, float *part, void *out, size_t ldo, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    if (splits == 0 || splits > KV_MAX_SPLITS) return fail(CERA_CUDA_ERR_BAD_ARG, "attention: %u splits", splits);
    return f32 ? grouped_attention<float>(q32, s, cache_k, cache_v, ld_v, n, start_pos, len_dev, splits, part, out, ldo, st)
               : grouped_attention<bf16>(q32, s, cache_k, cache_v, ld_v, n, start_pos, len_dev, splits, part, out, ldo, st);
}

}  // namespace cera
