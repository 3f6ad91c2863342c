// The state-space recurrence over a prompt portion in chunks of 64 tokens, on the tensor cores.  Inside a chunk, with L the
// running sum of the log decays and S the state the chunk starts from,
//   y_t = exp(L_t) S^T C_t + sum over j <= t of (C_t . B_j) exp(L_t - L_j) dt_j x_j + D x_t
//   S  <- exp(L_end) S + sum over j of B_j (exp(L_end - L_j) dt_j x_j)^T
// A CTA walks the chunks of one head (64 of its values).  Eight warps compute: a warp owns 16 values and half the rows of the
// state, whose f32 accumulators stay in registers from chunk to chunk and turn into operands of the first product as they
// are; the two halves of S^T C are exchanged through shared memory, each warp finishing two of the four 16-token tiles.  A
// ninth warp works out the next chunk's decays meanwhile.  B, C and x are bf16 as the convolution leaves them; decays, weights
// and states, f32, enter a product as a high and a low bf16 part.  L is summed in double and kept as two floats, so that
// close differences of large sums stay exact.
#include "mma.cuh"
#include "ssm.cuh"

namespace cera {

namespace {

constexpr int SC_Q = 64, SC_P = 64, SC_WARPS = 8, SC_LD = SC_P + 8;

template <int NT>  // the state's rows / 16
struct ChunkSmem {
    static constexpr int N = NT * 16, LD = N + 8;
    bf16 b[2][SC_Q][LD], c[2][SC_Q][LD], x[2][SC_Q][SC_LD];
    bf16 m[2][SC_Q][SC_LD], wx[2][SC_Q][SC_LD];  // high, low
    float4 half[SC_WARPS][4][32];  // of S^T C, for the warp that finishes the tile
    float l_hi[2][SC_Q], l_lo[2][SC_Q], dt[2][SC_Q], w[2][SC_Q], e[2][SC_Q];
    float e_end[2];
};

template <int NT>
__global__ void __launch_bounds__((SC_WARPS + 1) * 32) ssm_chunk_kernel(const float *pre, const bf16 *xbc, SsmView v, uint32_t n, uint32_t start_pos, float *y) {
    using Smem = ChunkSmem<NT>;
    constexpr int H = NT / 2;  // 16-row tiles of a warp's half of the state
    extern __shared__ __align__(16) uint8_t raw[];
    Smem &sm = *reinterpret_cast<Smem *>(raw);
    const SsmShape &s = v.s;
    pdl_trigger();
    const uint32_t h = blockIdx.x, g = h / (s.heads / s.groups), p0 = blockIdx.y * SC_P, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, N = s.state_p;
    const uint32_t width = min((uint32_t)SC_P, s.dim_p - p0), channels = s.channels(), r = lane >> 2, c2 = (lane & 3) * 2;
    const uint32_t pw = (warp & 3) * 16, nh = warp >> 2 & 1, n0 = nh * H * 16;  // this warp's values and rows
    const float rate = -expf(v.a_log[h]), dt_bias = v.dt_bias[h], dd = v.d[h];
    pdl_wait();
    auto decays = [&](uint32_t t0, int stage) {  // of the chunk at t0, by one warp: tokens 2 lane, 2 lane + 1
        float dt[2];
        double l[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint32_t t = t0 + 2 * lane + i;
            dt[i] = t < n ? softplus_f32(pre[(size_t)t * s.in_p + s.off_dt() + h] + dt_bias) : 0.0f;  // no token: nothing decays, nothing enters
            l[i] = (double)(rate * dt[i]);
        }
        l[1] += l[0];
        double before = l[1];
#pragma unroll
        for (int o = 1; o < 32; o *= 2) {
            const double u = __shfl_up_sync(0xffffffffu, before, o);
            if (lane >= (uint32_t)o) before += u;
        }
        const double end = __shfl_sync(0xffffffffu, before, 31);
        before -= l[1];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const double d = before + l[i];
            const uint32_t t = 2 * lane + i;
            sm.l_hi[stage][t] = (float)d;
            sm.l_lo[stage][t] = (float)(d - (double)(float)d);
            sm.dt[stage][t] = dt[i];
            sm.w[stage][t] = expf((float)(end - d)) * dt[i];
            sm.e[stage][t] = expf((float)d);
        }
        if (lane == 0) sm.e_end[stage] = expf((float)end);
    };
    if (warp == SC_WARPS) {
        decays(0, 0);
        int stage = 0;
        for (uint32_t t0 = 0; t0 < n; t0 += SC_Q, stage ^= 1) {
            __syncthreads();
            if (t0 + SC_Q < n) decays(t0 + SC_Q, stage ^ 1);
            __syncthreads();
        }
        return;
    }
    const bool owner = pw < width;
    // the state: value p0 + pw + r (+ 8), rows n0 + 8 i + c2 (+ 1)
    float S[2 * H][4];
    float *st = v.state + ((size_t)h * N + n0) * s.dim_p + p0 + pw + r;
#pragma unroll
    for (int i = 0; i < 2 * H; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const uint32_t row = i * 8 + c2 + (e & 1);
            S[i][e] = owner && n0 + row < N ? st[(size_t)row * s.dim_p + (e >> 1) * 8] : 0.0f;
        }
    auto fetch = [&](uint32_t t0, int stage) {
        auto rows = [&](bf16 *dst, uint32_t ld, uint32_t vecs, uint32_t live, uint32_t from) {
            for (uint32_t i = threadIdx.x; i < SC_Q * vecs; i += SC_WARPS * 32) {
                const uint32_t t = i / vecs, c = i - t * vecs;
                bf16 *d = dst + (size_t)t * ld + c * 8;
                if (t0 + t < n && c * 8 < live) tma::cp_async16(d, xbc + (size_t)(t0 + t) * channels + from + c * 8);
                else *reinterpret_cast<uint4 *>(d) = make_uint4(0, 0, 0, 0);
            }
        };
        rows(&sm.b[stage][0][0], Smem::LD, Smem::N / 8, N, s.off_b() + g * N);
        rows(&sm.c[stage][0][0], Smem::LD, Smem::N / 8, N, s.off_c() + g * N);
        rows(&sm.x[stage][0][0], SC_LD, SC_P / 8, width, h * s.dim_p + p0);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    const uint32_t k_row = (lane & 7) + ((lane >> 3) & 1) * 8, k_col = (lane >> 4) * 8;  // of a transposed 16 x 16 operand tile
    // token tiles: the first two this warp finishes, the others its partner; five tiles of M either way
    const uint32_t mts[4] = {nh ? 1u : 0u, nh ? 2u : 3u, nh ? 0u : 1u, nh ? 3u : 2u};
    int stage = 0;
    for (uint32_t t0 = 0; t0 < n; t0 += SC_Q, stage ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (t0 + SC_Q < n) fetch(t0 + SC_Q, stage ^ 1);
        const bf16 *bs = &sm.b[stage][0][0], *cs = &sm.c[stage][0][0], *xs = &sm.x[stage][0][0];
        const float *l_hi = sm.l_hi[stage], *l_lo = sm.l_lo[stage], *dts = sm.dt[stage], *ws = sm.w[stage], *es = sm.e[stage];
        // M: C_t . B_j with its weight, for the ten 16 x 16 tiles on and below the diagonal
#pragma unroll 1
        for (uint32_t tile = warp; tile < 10; tile += SC_WARPS) {
            const uint32_t mt = tile < 1 ? 0 : tile < 3 ? 1 : tile < 6 ? 2 : 3, nt = tile - mt * (mt + 1) / 2;
            const bf16 *ca = cs + (size_t)(mt * 16 + (lane & 15)) * Smem::LD + (lane >> 4) * 8;
            const bf16 *bb = bs + (size_t)(nt * 16 + (lane & 7) + (lane >> 4) * 8) * Smem::LD + ((lane >> 3) & 1) * 8;
            float gt[2][4] = {};
#pragma unroll
            for (int kk = 0; kk < NT; ++kk) {
                uint32_t a[4], b[4];
                ldsm4(a, ca + kk * 16);
                ldsm4(b, bb + kk * 16);
                mma_bf16(gt[0], a, b[0], b[1]);
                mma_bf16(gt[1], a, b[2], b[3]);
            }
#pragma unroll
            for (int q = 0; q < 2; ++q)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const uint32_t t = mt * 16 + r + 8 * i, j = nt * 16 + q * 8 + c2;
                    float m[2];
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        m[e] = j + e <= t ? gt[q][2 * i + e] * expf((l_hi[t] - l_hi[j + e]) + (l_lo[t] - l_lo[j + e])) * dts[j + e] : 0.0f;
                    uint32_t hi, lo;
                    split_bf16(m[0], m[1], hi, lo);
                    *reinterpret_cast<uint32_t *>(&sm.m[0][t][j]) = hi;
                    *reinterpret_cast<uint32_t *>(&sm.m[1][t][j]) = lo;
                }
        }
#pragma unroll
        for (int k = 0; k < SC_Q * SC_P / 2 / (SC_WARPS * 32); ++k) {
            const uint32_t i = threadIdx.x + k * SC_WARPS * 32, t = i / (SC_P / 2), p = i % (SC_P / 2) * 2;
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(xs + (size_t)t * SC_LD + p));
            uint32_t hi, lo;
            split_bf16(ws[t] * x.x, ws[t] * x.y, hi, lo);
            *reinterpret_cast<uint32_t *>(&sm.wx[0][t][p]) = hi;
            *reinterpret_cast<uint32_t *>(&sm.wx[1][t][p]) = lo;
        }
        // this half of S^T C
        float acc[4][2][4] = {};
        if (owner) {
            const bf16 *ca = cs + (size_t)(lane & 15) * Smem::LD + n0 + (lane >> 4) * 8;
#pragma unroll
            for (int kk = 0; kk < H; ++kk) {
                uint32_t sh[2][2], sl[2][2];  // [values][first or second eight rows]
#pragma unroll
                for (int q = 0; q < 2; ++q)
#pragma unroll
                    for (int u = 0; u < 2; ++u) split_bf16(S[2 * kk + u][2 * q], S[2 * kk + u][2 * q + 1], sh[q][u], sl[q][u]);
                uint32_t a[4][4];
#pragma unroll
                for (int o = 0; o < 4; ++o) ldsm4(a[o], ca + (size_t)mts[o] * 16 * Smem::LD + kk * 16);
#pragma unroll
                for (int o = 0; o < 4; ++o) {
                    mma_bf16(acc[o][0], a[o], sh[0][0], sh[0][1]);
                    mma_bf16(acc[o][1], a[o], sh[1][0], sh[1][1]);
                }
#pragma unroll
                for (int o = 0; o < 4; ++o) {
                    mma_bf16(acc[o][0], a[o], sl[0][0], sl[0][1]);
                    mma_bf16(acc[o][1], a[o], sl[1][0], sl[1][1]);
                }
            }
#pragma unroll
            for (int k = 0; k < 4; ++k)
                sm.half[warp ^ 4][k][lane] = make_float4(acc[2 + (k >> 1)][k & 1][0], acc[2 + (k >> 1)][k & 1][1], acc[2 + (k >> 1)][k & 1][2], acc[2 + (k >> 1)][k & 1][3]);
        }
        __syncthreads();
        if (!owner) continue;
        // the partner's last two tiles are this warp's first two, in the same order
#pragma unroll
        for (int o = 0; o < 2; ++o) {
            const float f0 = es[mts[o] * 16 + r], f1 = es[mts[o] * 16 + r + 8];
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                const float4 u = sm.half[warp][2 * o + q][lane];
                acc[o][q][0] = (acc[o][q][0] + u.x) * f0;
                acc[o][q][1] = (acc[o][q][1] + u.y) * f0;
                acc[o][q][2] = (acc[o][q][2] + u.z) * f1;
                acc[o][q][3] = (acc[o][q][3] + u.w) * f1;
            }
        }
#pragma unroll
        for (uint32_t kt = 0; kt < 4; ++kt) {
            uint32_t b[4];
            ldsm4_trans(b, xs + (size_t)(kt * 16 + k_row) * SC_LD + pw + k_col);
#pragma unroll
            for (int o = 0; o < 2; ++o) {
                if (kt > mts[o]) continue;
                uint32_t a[2][4];
#pragma unroll
                for (int part = 0; part < 2; ++part) ldsm4(a[part], &sm.m[part][mts[o] * 16 + (lane & 15)][kt * 16 + (lane >> 4) * 8]);
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    mma_bf16(acc[o][0], a[part], b[0], b[1]);
                    mma_bf16(acc[o][1], a[part], b[2], b[3]);
                }
            }
        }
#pragma unroll
        for (int o = 0; o < 2; ++o)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const uint32_t t = mts[o] * 16 + r + 8 * i;
                if (t0 + t >= n) continue;
#pragma unroll
                for (int q = 0; q < 2; ++q) {
                    const uint32_t p = pw + q * 8 + c2;
                    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(xs + (size_t)t * SC_LD + p));
                    *reinterpret_cast<float2 *>(y + (size_t)(t0 + t) * s.inner_p() + h * s.dim_p + p0 + p) =
                        make_float2(fmaf(dd, x.x, acc[o][q][2 * i]), fmaf(dd, x.y, acc[o][q][2 * i + 1]));
                }
            }
        const float end = sm.e_end[stage];
#pragma unroll
        for (int i = 0; i < 2 * H; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[i][e] *= end;
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {
            uint32_t ah[4], al[4], b[H][4];
            const uint32_t row = kt * 16 + (lane & 7) + (lane >> 4) * 8, col = pw + ((lane >> 3) & 1) * 8;
            ldsm4_trans(ah, &sm.wx[0][row][col]);
            ldsm4_trans(al, &sm.wx[1][row][col]);
#pragma unroll
            for (int i = 0; i < H; ++i) ldsm4_trans(b[i], bs + (size_t)(kt * 16 + k_row) * Smem::LD + n0 + i * 16 + k_col);
#pragma unroll
            for (int i = 0; i < H; ++i) {
                mma_bf16(S[2 * i], ah, b[i][0], b[i][1]);
                mma_bf16(S[2 * i + 1], ah, b[i][2], b[i][3]);
            }
#pragma unroll
            for (int i = 0; i < H; ++i) {
                mma_bf16(S[2 * i], al, b[i][0], b[i][1]);
                mma_bf16(S[2 * i + 1], al, b[i][2], b[i][3]);
            }
        }
    }
    if (owner) {
#pragma unroll
        for (int i = 0; i < 2 * H; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t row = i * 8 + c2 + (e & 1);
                if (n0 + row < N) st[(size_t)row * s.dim_p + (e >> 1) * 8] = S[i][e];
            }
    }
    ssm_keep(pre, v, h, p0, p0 + width, blockIdx.y == 0, n, start_pos, SC_WARPS * 32);
}

template <int NT>
int32_t launch_nt(const float *pre, const bf16 *xbc, const SsmView &v, size_t n, size_t start_pos, float *y, cudaStream_t st) {
    const dim3 grid(v.s.heads, (v.s.dim_p + SC_P - 1) / SC_P);
    auto k = ssm_chunk_kernel<NT>;
    CERA_CUDA_TRY(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, sizeof(ChunkSmem<NT>)));
    count_launch();
    return check_cuda(launch_k(k, grid, dim3((SC_WARPS + 1) * 32), sizeof(ChunkSmem<NT>), st, pre, xbc, v, (uint32_t)n, (uint32_t)start_pos, y), "ssm chunk launch");
}

}  // namespace

bool ssm_chunks_support(const SsmShape &s) { return s.state_p <= 256; }

int32_t launch_ssm_chunks(const float *pre, const void *xbc, const SsmView &v, size_t n, size_t start_pos, float *y, cudaStream_t st) {
    if (n == 0) return CERA_CUDA_OK;
    const bf16 *x = (const bf16 *)xbc;
    const uint32_t N = v.s.state_p;
    if (!ssm_chunks_support(v.s)) return fail(CERA_CUDA_ERR_UNSUPPORTED, "state-space chunks: state of %u", N);
    if (N <= 32) return launch_nt<2>(pre, x, v, n, start_pos, y, st);
    if (N <= 64) return launch_nt<4>(pre, x, v, n, start_pos, y, st);
    if (N <= 128) return launch_nt<8>(pre, x, v, n, start_pos, y, st);
    return launch_nt<16>(pre, x, v, n, start_pos, y, st);
}

}  // namespace cera
