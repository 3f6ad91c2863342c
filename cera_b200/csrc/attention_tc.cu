// Causal attention of a prompt portion on tcgen05: over the expanded keys and values of latent attention, or over the
// cached keys and values of grouped heads.
//
// A CTA owns 128 queries of one head and walks tiles of 64 keys: S = Q K^T (a part against the head's or group's own keys
// and, with latent attention, the rotated part against the shared rotated key; one accumulator), softmax on the CUDA cores in
// f32, O += P V with P as a bf16 operand in shared memory and V stored transposed.  One thread loads by TMA, one issues
// MMAs, four warps do the softmax (thread = query).  S and P are double-buffered so that the next tile's scores are formed
// during this tile's softmax.  O stays in TMEM and is rescaled only when a row's maximum has grown by more than 2^8.
// Scores may be soft-capped.  A sink enters the denominator at the end; a head's gate multiplies the stored output (both
// optional).  Every wait is bounded.
#include "dense.cuh"
#include "tc.cuh"
#include "tensor_map.h"

namespace cera {

__device__ unsigned int g_attention_tc_status = 0;

static const bool g_attention_tc_registered = register_kernel_status([] {
    unsigned int v = 0;
    cudaMemcpyFromSymbol(&v, g_attention_tc_status, sizeof(v));
    return (uint32_t)v << 20;
});

namespace {

constexpr int AT_Q = 128, AT_K = 64, AT_THREADS = 6 * 32;
constexpr uint32_t AT_QBLK = AT_Q * 128, AT_KBLK = AT_K * 128;  // bytes of a 64-column block of Q / K
constexpr uint32_t AT_P_BYTES = AT_Q * AT_K * 2;
constexpr float LOG2E = 1.44269504088896340736f;
constexpr float RESCALE_LOG2 = 8.0f;

struct AtParams {
    AttentionTcShape s;
    uint32_t n, start_pos, q_tiles, nb_dim, nb_rot;  // nb: 64-column blocks of the unrotated and the rotated part
    size_t ldo;
    const float *sink, *gate;
    bf16 *out;
};

__host__ __device__ inline uint32_t at_smem(const AttentionTcShape &s) {
    const uint32_t nb = (s.dim_p + 63) / 64 + (s.rot_p + 63) / 64;
    return 1024 + nb * AT_QBLK + 2 * AT_P_BYTES + 2 * (nb * AT_KBLK + s.vdim_p * 128) + 256;
}

__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <bool CAP>
__global__ void __launch_bounds__(AT_THREADS, 1) attention_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                                                       const __grid_constant__ CUtensorMap map_r, const __grid_constant__ CUtensorMap map_v,
                                                                       AtParams p) {
    extern __shared__ uint8_t raw[];
    const AttentionTcShape &s = p.s;
    const uint32_t nb = p.nb_dim + p.nb_rot, k_stage = nb * AT_KBLK, v_stage = s.vdim_p * 128;
    uint8_t *qs = raw + (1024 - (tma::smem_u32(raw) & 1023)) % 1024, *ps = qs + nb * AT_QBLK, *ks = ps + 2 * AT_P_BYTES, *vs = ks + 2 * k_stage;
    uint64_t *bars = reinterpret_cast<uint64_t *>(vs + 2 * v_stage);
    uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = bars + 3, *v_full = bars + 5, *v_empty = bars + 7, *s_full = bars + 9, *s_free = bars + 11,
             *p_full = bars + 13, *pv_done = bars + 15;
    uint32_t *tmem_at = reinterpret_cast<uint32_t *>(bars + 17);
    volatile uint32_t *abort_flag = tmem_at + 1;
    unsigned int *status = &g_attention_tc_status;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t h = blockIdx.x % s.heads, qt = p.q_tiles - 1 - blockIdx.x / s.heads, q0 = qt * AT_Q;  // longest rows first
    pdl_trigger();
    if (threadIdx.x == 0) {
        for (int i = 0; i < 17; ++i) tma::mbar_init(bars + i, i >= 11 && i < 15 ? 4 : 1);
        *abort_flag = 0;
        tma::mbar_init_fence();
    }
    if (warp == 1) {
        tmem_alloc(tmem_at, 512);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_at, tm_o = tmem + 2 * AT_K;
    pdl_wait();
    const uint32_t q_end = min(q0 + AT_Q, p.n), n_kv = (p.start_pos + q_end + AT_K - 1) / AT_K;
    const uint32_t hd = s.dim_p + s.rot_p, g = h / s.group;
    if (warp == 0) {
        if (lane == 0) {
            tma::mbar_expect_tx(q_full, nb * AT_QBLK);
            for (uint32_t b = 0; b < p.nb_dim; ++b) tma::tensor_g2s_2d(qs + b * AT_QBLK, &map_q, h * hd + b * 64, q0, q_full);
            for (uint32_t b = 0; b < p.nb_rot; ++b) tma::tensor_g2s_2d(qs + (p.nb_dim + b) * AT_QBLK, &map_q, h * hd + s.dim_p + b * 64, q0, q_full);
            uint32_t j = 0;
            for (; j < n_kv; ++j) {
                const uint32_t st = j & 1, par = (j >> 1 & 1) ^ 1;
                if (!tma::mbar_wait_blocking(k_empty + st, par, abort_flag, status, 1u)) break;
                uint8_t *kd = ks + st * k_stage;
                tma::mbar_expect_tx(k_full + st, k_stage);
                for (uint32_t b = 0; b < p.nb_dim; ++b) tma::tensor_g2s_2d(kd + b * AT_KBLK, &map_k, g * s.dim_p + b * 64, j * AT_K, k_full + st);
                for (uint32_t b = 0; b < p.nb_rot; ++b) tma::tensor_g2s_2d(kd + (p.nb_dim + b) * AT_KBLK, &map_r, b * 64, j * AT_K, k_full + st);
                if (!tma::mbar_wait_blocking(v_empty + st, par, abort_flag, status, 1u)) {
                    ++j;
                    break;
                }
                tma::mbar_expect_tx(v_full + st, v_stage);
                tma::tensor_g2s_2d(vs + st * v_stage, &map_v, j * AT_K, g * s.vdim_p, v_full + st);
            }
            if (*abort_flag) {  // this CTA's shared memory must outlive the copies in flight
                auto drain = [&](uint64_t *bar, uint32_t par) {
                    for (uint32_t n = 0; n < tma::SPIN_LIMIT && !tma::mbar_test(bar, par); ++n) __nanosleep(40);
                };
                drain(q_full, 0);
                for (uint32_t i = j > 2 ? j - 2 : 0; i < j; ++i) {
                    drain(k_full + (i & 1), i >> 1 & 1);
                    if (i + 1 < j) drain(v_full + (i & 1), i >> 1 & 1);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t id_s = tc_idesc_bf16(AT_Q, AT_K), id_o = tc_idesc_bf16(AT_Q, s.vdim_p);
            auto scores = [&](uint32_t j) -> bool {
                const uint32_t b = j & 1, par = j >> 1 & 1;
                if (!tma::mbar_wait_blocking(k_full + b, par, abort_flag, status, 2u)) return false;
                if (!tma::mbar_wait_blocking(s_free + b, par ^ 1, abort_flag, status, 2u)) return false;
                tc_fence_after();
                const uint32_t qa = tma::smem_u32(qs), ka = tma::smem_u32(ks + b * k_stage);
                uint32_t acc = 0;
                for (uint32_t part = 0; part < 2; ++part) {
                    const uint32_t steps = (part ? s.rot_p : s.dim_p) / 16, blk0 = part ? p.nb_dim : 0;
                    for (uint32_t k = 0; k < steps; ++k, acc = 1) {
                        const uint32_t blk = blk0 + (k >> 2), kk = k & 3;
                        tc_mma_f16(tmem + b * AT_K, smem_desc_sw128(qa + blk * AT_QBLK) + 2 * kk, smem_desc_sw128(ka + blk * AT_KBLK) + 2 * kk, id_s, acc);
                    }
                }
                tc_commit(k_empty + b);
                tc_commit(s_full + b);
                return true;
            };
            bool ok = tma::mbar_wait_blocking(q_full, 0, abort_flag, status, 2u) && scores(0);
            for (uint32_t j = 0; j < n_kv && ok; ++j) {
                if (j + 1 < n_kv && !(ok = scores(j + 1))) break;
                const uint32_t b = j & 1, par = j >> 1 & 1;
                ok = tma::mbar_wait_blocking(p_full + b, par, abort_flag, status, 2u) && tma::mbar_wait_blocking(v_full + b, par, abort_flag, status, 2u);
                if (!ok) break;
                tc_fence_after();
                const uint32_t pa = tma::smem_u32(ps + b * AT_P_BYTES), va = tma::smem_u32(vs + b * v_stage);
#pragma unroll
                for (int k = 0; k < AT_K / 16; ++k) tc_mma_f16(tm_o, smem_desc_sw128(pa) + 2 * k, smem_desc_sw128(va) + 2 * k, id_o, j | k);
                tc_commit(v_empty + b);
                tc_commit(pv_done + b);
            }
        }
    } else {
        const uint32_t quad = warp & 3, r = quad * 32 + lane, lanes = quad * 32 << 16, pos = p.start_pos + q0 + r;
        // a score in units of ln 2: the product times sc2, or cap tanh(product / cap) with tanh(z) = 1 - 2 / (1 + e^2z)
        const float sc2 = CAP ? 2.0f * LOG2E * s.scale / s.softcap : s.scale * LOG2E, cap2 = s.softcap * LOG2E;
        auto score = [&](uint32_t bits) {
            const float z = __uint_as_float(bits) * sc2;
            return CAP ? fmaf(-2.0f * cap2, rcp_approx(1.0f + exp2_approx(z)), cap2) : z;
        };
        float m = -INFINITY, l = 0.0f;
        bool ok = true;
        for (uint32_t j = 0; j < n_kv; ++j) {
            const uint32_t b = j & 1, par = j >> 1 & 1;
            ok = __all_sync(0xffffffffu, tma::mbar_wait_blocking(s_full + b, par, abort_flag, status, 4u));
            if (!ok) break;
            tc_fence_after();
            uint32_t v[4][16];
#pragma unroll
            for (int i = 0; i < 4; ++i) tmem_ld16(tmem + lanes + b * AT_K + i * 16, v[i]);
            tmem_wait_ld();
            tc_fence_before();
            if (lane == 0) tma::mbar_arrive(s_free + b);
            float x[AT_K], mx = -INFINITY;
            const uint32_t key0 = j * AT_K;
            if (key0 + AT_K - 1 > p.start_pos + q0) {  // some query of the tile does not see some key of this one
#pragma unroll
                for (int i = 0; i < AT_K; ++i) {
                    x[i] = key0 + i <= pos ? score(v[i >> 4][i & 15]) : -INFINITY;
                    mx = fmaxf(mx, x[i]);
                }
            } else {
#pragma unroll
                for (int i = 0; i < AT_K; ++i) {
                    x[i] = score(v[i >> 4][i & 15]);
                    mx = fmaxf(mx, x[i]);
                }
            }
            // every row sees key 0, so m is finite from the first tile on
            float alpha = 1.0f;
            if (mx > m + RESCALE_LOG2 || j == 0) {
                alpha = exp2_approx(m - mx);
                m = mx;
                l *= alpha;
            }
            if (j > 0) {
                if (__any_sync(0xffffffffu, alpha != 1.0f)) {  // O of the tiles before must be complete to be rescaled
                    ok = __all_sync(0xffffffffu, tma::mbar_wait_blocking(pv_done + (b ^ 1), (j - 1) >> 1 & 1, abort_flag, status, 4u));
                    if (!ok) break;
                    tc_fence_after();
                    for (uint32_t c = 0; c < s.vdim_p; c += 16) {
                        uint32_t o[16];
                        tmem_ld16(tm_o + lanes + c, o);
                        tmem_wait_ld();
#pragma unroll
                        for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                        tmem_st16(tm_o + lanes + c, o);
                    }
                    tmem_wait_st();
                }
                if (j > 1) {  // P of two tiles ago has been read
                    ok = __all_sync(0xffffffffu, tma::mbar_wait_blocking(pv_done + b, (j - 2) >> 1 & 1, abort_flag, status, 4u));
                    if (!ok) break;
                }
            }
            uint8_t *row = ps + b * AT_P_BYTES + r * 128;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                uint32_t w[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float e0 = exp2_approx(x[c * 8 + 2 * i] - m), e1 = exp2_approx(x[c * 8 + 2 * i + 1] - m);
                    l += e0 + e1;
                    const __nv_bfloat162 pr = __floats2bfloat162_rn(e0, e1);
                    w[i] = *reinterpret_cast<const uint32_t *>(&pr);
                }
                *reinterpret_cast<uint4 *>(row + ((c ^ (r & 7)) << 4)) = make_uint4(w[0], w[1], w[2], w[3]);
            }
            fence_async_smem();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) tma::mbar_arrive(p_full + b);
        }
        if (ok) ok = __all_sync(0xffffffffu, tma::mbar_wait_blocking(pv_done + ((n_kv - 1) & 1), (n_kv - 1) >> 1 & 1, abort_flag, status, 4u));
        if (ok) {
            tc_fence_after();
            const bool live = q0 + r < p.n;
            if (p.sink) l += exp2_approx(p.sink[h] * LOG2E - m);
            const float f = live ? (p.gate ? p.gate[(size_t)(q0 + r) * s.heads + h] : 1.0f) / l : 0.0f;
            for (uint32_t c = 0; c < s.vdim_p; c += 16) {
                uint32_t o[16];
                tmem_ld16(tm_o + lanes + c, o);
                tmem_wait_ld();
                uint32_t w[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const __nv_bfloat162 pr = __floats2bfloat162_rn(__uint_as_float(o[2 * i]) * f, __uint_as_float(o[2 * i + 1]) * f);
                    w[i] = *reinterpret_cast<const uint32_t *>(&pr);
                }
                if (live) {
                    uint4 *dst = reinterpret_cast<uint4 *>(p.out + (size_t)(q0 + r) * p.ldo + h * s.vdim_p + c);
                    dst[0] = make_uint4(w[0], w[1], w[2], w[3]);
                    dst[1] = make_uint4(w[4], w[5], w[6], w[7]);
                }
            }
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, 512);
}

}  // namespace

bool attention_tc_supports(const AttentionTcShape &s) { return s.vdim_p <= 256 && at_smem(s) <= 227 * 1024; }

int32_t launch_attention_tc(const AttentionTcShape &s, const AttentionTcOperands &o, size_t n, size_t start_pos, void *out, size_t ldo, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    if (!attention_tc_supports(s)) return fail(CERA_CUDA_ERR_UNSUPPORTED, "prompt attention: heads of %u + %u / %u", s.dim_p, s.rot_p, s.vdim_p);
    const uint64_t total = start_pos + n, kv_heads = s.heads / s.group;
    if (total > o.positions || total > o.ld_v) return fail(CERA_CUDA_ERR_BAD_ARG, "prompt attention: %zu positions", (size_t)total);
    CUtensorMap mq, mk, mr, mv;
    CERA_TRY(tensor_map_bf16(&mq, o.q, n, (uint64_t)s.heads * (s.dim_p + s.rot_p), 64, AT_Q));
    CERA_TRY(tensor_map_bf16(&mk, o.k, total, kv_heads * s.dim_p, 64, AT_K));
    if (s.rot_p) CERA_TRY(tensor_map_bf16(&mr, o.k_rot, total, s.rot_p, 64, AT_K));
    else mr = mk;  // not used
    CERA_TRY(tensor_map_bf16(&mv, o.v, kv_heads * s.vdim_p, o.ld_v, 64, s.vdim_p));
    AtParams p;
    p.s = s;
    p.n = (uint32_t)n;
    p.start_pos = (uint32_t)start_pos;
    p.q_tiles = (uint32_t)((n + AT_Q - 1) / AT_Q);
    p.nb_dim = (s.dim_p + 63) / 64;
    p.nb_rot = (s.rot_p + 63) / 64;
    p.ldo = ldo;
    p.sink = o.sink;
    p.gate = o.gate;
    p.out = (bf16 *)out;
    auto kernel = s.softcap > 0.0f ? attention_tc_kernel<true> : attention_tc_kernel<false>;
    CERA_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    count_launch();
    return check_cuda(launch_k(kernel, dim3(p.q_tiles * s.heads), dim3(AT_THREADS), at_smem(s), st, mq, mk, mr, mv, p), "prompt attention launch");
}

}  // namespace cera
