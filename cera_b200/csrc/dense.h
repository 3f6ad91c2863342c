// Dense (bf16 or f32) weights and the operators of models described layer by layer (layered.cu).
//
// Conventions: activations are token-major rows; T, the element type of weights and activations, is bf16 or f32
// (`f32` flags); every row length `ld` is a multiple of 64 elements and the padding is zero, so kernels walk whole
// 16-byte vectors and padded weight rows produce zeros.  Residual stream, norms, routing, scores, recurrent state: f32.
#pragma once

#include <cuda_bf16.h>

#include "ops.h"

namespace cera {

struct DenseView {
    const void *w = nullptr;
    uint32_t rows = 0, ld = 0;  // [rows][ld], zero-padded
    int f32 = 0;
};

inline uint32_t pad_to(uint32_t v, uint32_t a) { return (v + a - 1) / a * a; }

// A norm: g holds one number (per_channel 0) or one per channel (1, the row length's padding included).
struct NormView {
    const float *g = nullptr;
    int per_channel = 0;
    __device__ __forceinline__ float4 at(uint32_t i4) const {  // of channels 4 i4 .. 4 i4 + 3
        if (per_channel) return reinterpret_cast<const float4 *>(g)[i4];
        const float v = *g;
        return make_float4(v, v, v, v);
    }
};

// Index i of a padded axis: groups of `group` source entries become groups of `group_p`, of which the first `seg`
// entries stay in front and the rest start at seg_p.
struct PadMap {
    uint32_t group = 0xFFFFFFFFu, group_p = 0, seg = 0xFFFFFFFFu, seg_p = 0, base = 0;
    __host__ __device__ uint32_t operator()(uint32_t i) const {
        const uint32_t g = i / group, r = i - g * group;
        return base + g * group_p + (r < seg ? r : seg_p + (r - seg));
    }
};

// ---- weights (dense.cu) ---------------------------------------------------------------------------------------
// src [rows][cols] of CERA_TYPE_BF16 / F16 / F32, plus offset -> dst element (rmap(row), cmap(col)) of row length ld.
int32_t launch_place(const void *src, int32_t src_type, size_t rows, size_t cols, void *dst, int dst_f32, size_t ld, const PadMap &rmap,
                     const PadMap &cmap, cudaStream_t st, float offset = 0.0f);

// ---- embedding and norms (dense.cu) ------------------------------------------------------------------------------
struct BigramParams {
    uint32_t buckets = 0;  // 0: none
    uint64_t mul_prev = 0, mul_cur = 0;
};
// x[j] = table[token j] * scale (+ bigram row), also into `keep` when given.  tokens[0] is the token before the first one (NO_TOKEN: none), tokens[1 + j] token
// j; with dyn the step's token and its predecessor are read from the dyn words instead (n == 1).
int32_t launch_embed_dense(const DenseView &table, const DenseView &bigram, const BigramParams &bp, const uint32_t *tokens, const uint32_t *dyn,
                           size_t n, float scale, float *x, float *keep, cudaStream_t st);
// One sublayer boundary for n rows of `width` numbers (row length ld):
//   y (optional): x += norm_post(sum over picks of y[entry]) with entry = entry_of[j * picks + s], or row j without it
//     (post.g null: the sum itself); x += add[j] (optional);
//   then h = norm_pre(x), as T in h and / or f32 in h32.
// x_rows (optional): row j of x is x[x_rows[j]] (no residual update then).
struct ResidualNorm {
    float *x = nullptr;
    const float *y = nullptr;
    const uint32_t *entry_of = nullptr;
    const float *pick_weight = nullptr;  // multiplies an entry's row
    uint32_t picks = 1;
    const float *add = nullptr;
    NormView post, pre;
    void *h = nullptr;
    int h_f32 = 0;
    float *h32 = nullptr;
    const uint32_t *x_rows = nullptr;
};
int32_t launch_residual_norm(const ResidualNorm &p, uint32_t width, uint32_t ld, size_t n, float eps, cudaStream_t st);

// ---- one-column products (dense_gemv.cu) --------------------------------------------------------------------------
int32_t launch_dense_gemv(const DenseView &w, const void *x, float *y, cudaStream_t st);
// minGRU decode step: rows [0, wp) z, [wp, 2 wp) candidate, [2 wp, 3 wp) gate of w; updates state, out = state * silu(gate).
int32_t launch_mingru_step(const DenseView &w, const void *x, const float *z_bias, const float *x_bias, float *state, void *out, cudaStream_t st);
// A gated unit: min(g, limit) * sigmoid(alpha g) * (clamp(u, +-limit) + shift); limit inf, alpha 1, shift 0: silu(g) u.
struct ExpertAct {
    float limit = 0.0f, alpha = 0.0f, shift = 0.0f;
};
// Rows [0, ff_p) gate, [ff_p, 2 ff_p) up of w; out [ff_p] of T = unit(gate, up).
int32_t launch_gated_unit_step(const DenseView &w, const void *x, const ExpertAct &a, void *out, cudaStream_t st);
struct RouterRule {
    uint32_t n_expert = 0, n_used = 0;
    int softmax = 0, renorm = 0, weight_input = 0;
};
// Routed feed-forward of one token: picks from the router logits, gate / up rows of the chosen experts through the gated
// unit into act [n_used][ff_p]; the second call y = sum over picks of down rows.  w_gate_up stacks per expert ff_p gate
// rows then ff_p up rows, w_down `rows_per_expert` rows per expert.
int32_t launch_expert_gate_up_step(const DenseView &w_gate_up, const void *x, const float *router_logits, const RouterRule &r, uint32_t ff_p,
                                   const ExpertAct &a, uint32_t *ids, float *weights, void *act, cudaStream_t st);
int32_t launch_expert_down_step(const DenseView &w_down, uint32_t rows_per_expert, const void *act, const RouterRule &r, const uint32_t *ids,
                                const float *weights, float *y, cudaStream_t st);

// ---- many-column products (dense_gemm.cu, dense_gemm_tc.cu) ----------------------------------------------------------
enum DenseOut { DENSE_F32 = 0, DENSE_T = 1, DENSE_T_TRANSPOSED = 2, DENSE_GATED_UNIT = 3 };
struct DenseGemm {
    DenseView w;
    const void *x = nullptr;  // [n][w.ld]
    uint32_t n = 0;           // rows of x (grouped: rows of the gathered buffer)
    int out_kind = DENSE_F32;
    void *out = nullptr;  // out[j * ldo + row]; transposed: out[row * ldo + j]
    size_t ldo = 0;
    // grouped by expert: item (expert, first, count) takes rows [expert * rows_per_expert, + rows_per_expert) of w against
    // columns [first, first + count)
    const MoeTile *tiles = nullptr;
    const uint32_t *n_tiles = nullptr;
    uint32_t max_tiles = 0, rows_per_expert = 0, group_columns = 0;  // group_columns: most columns of an item
    // DENSE_GATED_UNIT: rows_per_expert (not grouped: w.rows) = 2 ff_p, out [columns][ff_p] of T = unit(scale * gate, scale * up)
    ExpertAct act;
    const float *col_scale = nullptr;
    // block-diagonal (not grouped): rows [b * block_rows, + block_rows) of w meet columns [b * w.ld, + w.ld) of x, whose rows are
    // x_ld long; block_rows is a multiple of 128
    uint32_t block_rows = 0;
    uint32_t x_ld = 0;
    uint32_t row_len() const { return x_ld ? x_ld : w.ld; }
};
// Columns of a grouped item when `entries` columns spread over n_expert experts.
constexpr uint32_t DENSE_GROUP_MIN = 32;
inline uint32_t dense_group_columns(uint32_t entries, uint32_t n_expert) {
    const uint32_t avg = entries / n_expert;
    return avg <= 24 ? 32 : avg <= 48 ? 64 : 128;
}
int32_t launch_dense_gemm(const DenseGemm &g, cudaStream_t st);
// The bf16 product on tcgen05 / TMEM.  *taken = false: not its case, nothing launched.
int32_t launch_dense_gemm_tc(const DenseGemm &g, cudaStream_t st, bool *taken);
// Columns of a batch in bucket order: g[pos] = h[token], entry_of[pair] = pos, col_scale[pos] = the pair's weight.
int32_t launch_moe_gather(const void *h, int f32, uint32_t ld, const uint32_t *ids, const float *weights, uint32_t n_used, size_t n, uint32_t *cursor,
                          uint32_t *entry_of, void *g, float *col_scale, cudaStream_t st);

// ---- minGRU over a prompt portion (mingru.cu) -----------------------------------------------------------------------
// pre: [n][3 wp] raw z / candidate / gate products; state: [wp], advanced by n positions.
int32_t launch_mingru_scan(const float *pre, size_t n, uint32_t wp, const float *z_bias, const float *x_bias, float *state, void *out, int f32,
                           cudaStream_t st);

// ---- how a cache of n_positions is cut for one query: splits of 64 positions or more -------------------------------------
constexpr uint32_t KV_MAX_SPLITS = 128;
inline uint32_t kv_splits(size_t n_positions) {
    uint32_t s = 1;
    while (s < KV_MAX_SPLITS && s * 64 < n_positions) s *= 2;
    return s;
}

// ---- latent attention (latent_attention.cu) --------------------------------------------------------
struct LatentShape {
    uint32_t heads = 0, dim = 0, rot = 0, vdim = 0, rank = 0;          // as the model states them
    uint32_t dim_p = 0, rot_p = 0, vdim_p = 0, rank_p = 0, in_p = 0;    // padded; in_p: row length of the input products
    __host__ __device__ uint32_t q_ld() const { return heads * (dim_p + rot_p); }
    __host__ __device__ uint32_t off_c() const { return heads * (dim_p + rot_p); }
    __host__ __device__ uint32_t off_r() const { return off_c() + rank_p; }
    __host__ __device__ uint32_t off_g() const { return off_r() + rot_p; }
    float scale = 0.0f;
};
// Input products [n][in_p] = q | latent | rotated key | gate logits.  Normalises the latent, rotates the key part and q,
// appends both to the cache at positions pos.. (pos_dev: read from device memory, n == 1), q as f32 (q32) and / or T (qt),
// gate = sigmoid(logit) [n][heads].
int32_t launch_latent_prepare(const float *in, const LatentShape &s, size_t n, size_t start_pos, const uint32_t *pos_dev, const float *c_norm, float eps,
                              const float *rope_table, void *cache_c, void *cache_r, int f32, float *q32, void *qt, float *gate, cudaStream_t st);
// Attention in the latent space for n queries at positions start_pos + j (or *len_dev - 1): q_lat = W_uk^T q, scores
// against the cached latents, per-split partial sums, merge with the sink, W_uv, gate.  out [n][ldo] of T, heads * vdim_p used.
struct LatentScratch {
    float *q_lat = nullptr;  // [queries][heads][rank_p + rot_p] f32, or as many pairs of bf16
    float *part = nullptr;   // [queries][heads][splits][rank_p + 2]
};
constexpr uint32_t LATENT_MAX_SPLITS = KV_MAX_SPLITS;  // queries * splits of one call never exceed this
int32_t launch_latent_attention(const float *q32, const LatentShape &s, const DenseView &uk, const DenseView &uv, const void *cache_c, const void *cache_r,
                                const float *sink, const float *gate, size_t n, size_t start_pos, const uint32_t *len_dev, uint32_t splits,
                                const LatentScratch &ws, void *out, size_t ldo, cudaStream_t st);

// ---- prompt attention on the tensor cores (attention_tc.cu) ---------------------------------------------------------------
// Head h attends with its query [dim_p | rot_p] to key group h / group: keys [positions][groups * dim_p], with rot_p also a
// part [positions][rot_p] that all groups share, values transposed [groups * vdim_p][ld_v].  All bf16; padding is zero.
struct AttentionTcShape {
    uint32_t heads = 0, group = 1, dim_p = 0, rot_p = 0, vdim_p = 0;
    float scale = 0.0f, softcap = 0.0f;  // softcap 0: none
};
struct AttentionTcOperands {
    const void *q = nullptr, *k = nullptr, *k_rot = nullptr, *v = nullptr;
    size_t positions = 0, ld_v = 0;                // rows of k; row length of v
    const float *sink = nullptr, *gate = nullptr;  // per head; per (query, head); optional
};
bool attention_tc_supports(const AttentionTcShape &s);
// n queries at positions start_pos..; out [n][ldo] of bf16, heads * vdim_p used.
int32_t launch_attention_tc(const AttentionTcShape &s, const AttentionTcOperands &o, size_t n, size_t start_pos, void *out, size_t ldo, cudaStream_t st);

// ---- attention with grouped key / value heads (grouped_attention.cu) -------------------------------------------------------
struct GroupedShape {
    uint32_t heads = 0, kv_heads = 0, dim = 0, rot = 0, vdim = 0;  // as the model states them; rot: rotated dimensions, the first of a head
    uint32_t dim_p = 0, vdim_p = 0, in_p = 0;                      // padded; in_p: row length of the input products
    float scale = 0.0f, softcap = 0.0f, eps = 0.0f;
    int qk_norm = 0;
    __host__ __device__ uint32_t q_ld() const { return heads * dim_p; }
    __host__ __device__ uint32_t off_k() const { return heads * dim_p; }
    __host__ __device__ uint32_t off_v() const { return off_k() + kv_heads * dim_p; }
    __host__ __device__ uint32_t in_rows() const { return off_v() + kv_heads * vdim_p; }
};
// Input products [n][in_p] = q | k | v.  Adds the biases, rotates q and k, brings their heads to unit root mean square
// (qk_norm), appends k to cache_k [positions][kv_heads * dim_p] and v to cache_v [kv_heads * vdim_p][ld_v]; q as f32 (q32) and /
// or T (qt).  pos_dev: the position is read from device memory (n == 1).
int32_t launch_grouped_prepare(const float *in, const GroupedShape &s, size_t n, size_t start_pos, const uint32_t *pos_dev, const float *bias,
                               const float *rope_table, void *cache_k, void *cache_v, size_t ld_v, int f32, float *q32, void *qt, cudaStream_t st);
// n queries at positions start_pos + j (or *len_dev - 1) over the cache, cut into splits; part: scratch of
// n * heads * splits * (vdim_p + 2) numbers.  out [n][ldo] of T.
int32_t launch_grouped_attention(const float *q32, const GroupedShape &s, const void *cache_k, const void *cache_v, size_t ld_v, int f32, size_t n,
                                 size_t start_pos, const uint32_t *len_dev, uint32_t splits, float *part, void *out, size_t ldo, cudaStream_t st);

// ---- short causal convolution per channel (conv.cuh, conv.cu) ---------------------------------------------------------------
// value(t) = bias + sum over k of w[channel][k] * input(t - (taps - 1 - k)), inputs before the sequence are zero.
struct ConvView {
    const float *w = nullptr, *bias = nullptr;  // [channels][taps], [channels]
    float *ring = nullptr;  // [taps][channels]: the inputs of the last positions, position p in row p mod taps
    uint32_t channels = 0, taps = 0;
};
// Portion: in [n][ld_in] products of the positions start_pos.., in_bias (optional) is added to them; out [n][ld_out] of T,
// through silu or not.  Reads the ring and leaves it: conv_keep (conv.cuh) moves it on.
int32_t launch_conv(const float *in, size_t ld_in, const float *in_bias, const ConvView &c, int silu, size_t n, size_t start_pos, void *out, size_t ld_out,
                    int f32, cudaStream_t st);

// ---- real-gated linear recurrent unit (rglru.cu) ---------------------------------------------------------------------------
// The width is cut into blocks, each padded to block_p channels: wp = blocks * block_p.
struct RglruView {
    uint32_t wp = 0, block_p = 0;
    DenseView gates;  // per block block_p rows of the decay gate, block_p of the input gate; block_p columns
    const float *in_bias = nullptr;    // [2 wp]: of the output branch, of the convolved branch
    const float *gate_bias = nullptr;  // [2 wp]: as the rows of `gates`
    const float *lam = nullptr;        // [wp]
    float decay = 0.0f;                // log a = -decay * gate * softplus(lam)
    ConvView conv;
    float *state = nullptr;  // [wp]
};
// pre [2 wp]: products of the output branch and the convolved branch; out [wp] of T.
int32_t launch_rglru_step(const float *pre, const RglruView &v, const uint32_t *pos_dev, void *out, cudaStream_t st);
// A portion after launch_conv (u [n][wp] of T) and the gates' product (gate [n][2 wp] raw): out [n][wp] of T.
int32_t launch_rglru_scan(const float *pre, const void *u, const float *gate, const RglruView &v, size_t n, size_t start_pos, void *out, int f32,
                          cudaStream_t st);

// ---- state-space recurrence with a matrix state per head (ssm.cu, ssm_chunk.cu) --------------------------------------------
constexpr uint32_t SSM_MAX_STATE = 768;  // state_p at most (the scan's shared memory)
struct SsmShape {
    uint32_t heads = 0, dim = 0, state = 0, groups = 0, norm_groups = 0;  // dim: values of a head
    uint32_t dim_p = 0, state_p = 0, in_p = 0;                            // padded; in_p: row length of the input products
    float eps = 0.0f;
    // input products: z | x | B | C | step sizes; the convolution's channels are x | B | C
    __host__ __device__ uint32_t inner_p() const { return heads * dim_p; }
    __host__ __device__ uint32_t channels() const { return inner_p() + 2 * groups * state_p; }
    __host__ __device__ uint32_t off_b() const { return inner_p(); }  // among the channels
    __host__ __device__ uint32_t off_c() const { return inner_p() + groups * state_p; }
    __host__ __device__ uint32_t off_dt() const { return inner_p() + channels(); }  // among the products
    __host__ __device__ uint32_t in_rows() const { return off_dt() + heads; }
};
struct SsmView {
    SsmShape s;
    const float *dt_bias = nullptr, *a_log = nullptr, *d = nullptr;  // [heads]
    const float *norm = nullptr;                                      // [inner_p]
    ConvView conv;
    float *state = nullptr;  // [heads][state_p][dim_p]
};
// One position: convolution, state, y [inner_p] f32 (before gate and norm).
int32_t launch_ssm_step(const float *pre, const SsmView &v, const uint32_t *pos_dev, float *y, int f32, cudaStream_t st);
// A portion after launch_conv (xbc [n][channels] of T): y [n][inner_p].
int32_t launch_ssm_scan(const float *pre, const void *xbc, const SsmView &v, size_t n, size_t start_pos, float *y, int f32, cudaStream_t st);
// The same in chunks on the tensor cores (bf16).
bool ssm_chunks_support(const SsmShape &s);
int32_t launch_ssm_chunks(const float *pre, const void *xbc, const SsmView &v, size_t n, size_t start_pos, float *y, cudaStream_t st);
// out = rms_norm of each of norm_groups parts of (y * silu(z)), times the weight; out [n][ldo] of T.
int32_t launch_gated_norm(const float *y, const float *pre, const SsmView &v, size_t n, void *out, size_t ldo, int f32, cudaStream_t st);

}  // namespace cera
