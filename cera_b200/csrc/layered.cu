// A decoder described layer by layer: every layer names its token mixer (latent attention, minGRU) and its feed-forward
// (routed experts, or none), weights are dense (bf16 or f32).  A sublayer is normed before and after:
// x += post(sublayer(pre(x))), and the boundary between two sublayers - the residual sum of one, the norm of the next -
// is one kernel.
//
// Per sequence a latent-attention layer caches one latent and one rotated key part per position; a minGRU layer holds
// one f32 state vector; the bigram embedding needs the previous token (the base's history / dyn words).
//
// A decode step per layer: [boundary] -> minGRU: [z / candidate / gate products + state update] [output product];
// latent attention: [input products] [norm, rotation, cache append] [W_uk on the query] [split attention] [merge, W_uv, gate]
// [output product]; experts: [boundary] [router logits] [pick, gate / up, gated unit] [down, sum over picks].
// A prompt portion takes the same steps with many-column products, a scan for minGRU, and experts grouped by a device-built
// work list.
#include <cmath>
#include <cstring>
#include <new>
#include <vector>

#include "dense.h"
#include "model.h"

using namespace cera;

namespace {

constexpr size_t LAYERED_CHUNK = 2048;   // prompt tokens per chunk
constexpr size_t LATENT_EXPAND_MIN = 16;  // shorter portions attend in the latent space

struct ExpertFfn {
    DenseView gate_up, down, router;  // gate_up: per expert ff_p gate rows, ff_p up rows; router: f32
    uint32_t ff_p = 0;
};

struct LayerState {
    cera_cuda_layer_desc d{};
    LatentShape s;
    NormView pre, post, ff_pre, ff_post;
    DenseView in, out;  // the mixer's input products stacked into one matrix; its output projection
    // latent attention
    DenseView uk, uv;
    float *c_norm = nullptr, *sink = nullptr, *rope = nullptr;
    void *cache_c = nullptr, *cache_r = nullptr;
    // minGRU
    uint32_t wp = 0;
    float *z_bias = nullptr, *x_bias = nullptr, *state = nullptr;
    ExpertFfn ffn;
    std::vector<bool> seen;  // tensors given, by slot
};

enum Slot { S_PRE, S_POST, S_FF_PRE, S_FF_POST, S_OUT, S_A, S_B, S_C, S_D, S_E, S_F, S_G, S_ROUTER, S_EXPERTS };

struct LayeredModel : cera_cuda_model {
    LayeredModel(const cera_cuda_layered_config &c, const cera_cuda_layer_desc *l)
        : cera_cuda_model(c.vocab_size, c.hidden_size, c.max_seq_len, c.device), cfg(c), f32(c.dtype == CERA_TYPE_F32), esz(f32 ? 4 : 2),
          ld(pad_to(c.hidden_size, 64)), layers(c.n_layers) {
        for (uint32_t i = 0; i < c.n_layers; ++i) layers[i].d = l[i];
        bigram_rule.buckets = c.bigram_buckets;
        bigram_rule.mul_prev = c.bigram_mul_prev;
        bigram_rule.mul_cur = c.bigram_mul_cur;
    }
    int32_t place_layers();  // allocates the weights and works out the padded shapes
    int32_t add_tensor(int32_t role, int32_t layer, int32_t type, size_t rows, size_t cols, const void *bytes, size_t nbytes) override;
    int32_t add_expert(int32_t role, uint32_t layer, uint32_t expert, int32_t type, size_t rows, size_t cols, const void *bytes, size_t nbytes);
    int32_t build() override;
    size_t chunk_tokens() const override { return LAYERED_CHUNK; }
    uint32_t plan(size_t n_positions) const override { return has_attention ? latent_splits(n_positions) : 1; }
    int32_t enqueue_step(int kind, uint32_t splits) override;
    bool batched(size_t n) const override { return n >= 2; }
    int32_t prefill_chunk(const uint32_t *tokens, size_t n, size_t start_pos) override;
    int32_t logits_of_last(size_t n) override;
    int32_t logits_of_rows(const uint32_t *rows, size_t n_rows, size_t n, float *out) override;
    int32_t rewind(size_t len) override;
    size_t snapshot_bytes() const override;
    int32_t snapshot(void *out, size_t out_bytes) override;
    int32_t restore(const void *data, size_t bytes) override;

    int32_t dense(DenseView *v, uint32_t rows, uint32_t cols_p, int as_f32);
    int32_t vec(float **p, uint32_t n);
    int32_t place(const void *bytes, size_t nbytes, int32_t type, size_t rows, size_t cols, const DenseView &v, const PadMap &rmap, const PadMap &cmap);
    int32_t mixer_chunk(LayerState &L, size_t n, size_t start_pos, float *y);
    int32_t latent_chunk(LayerState &L, size_t n, size_t start_pos);
    int32_t experts_chunk(LayerState &L, size_t n, ResidualNorm *next);

    const cera_cuda_layered_config cfg;
    const int f32;
    const size_t esz;
    const uint32_t ld;
    BigramParams bigram_rule;
    bool has_attention = false, has_recurrence = false;
    DenseView embd, bigram, head;
    NormView out_norm;
    bool head_seen = false, embd_seen = false, bigram_seen = false;
    std::vector<LayerState> layers;
    // scratch; chunk buffers have LAYERED_CHUNK rows, the decode step uses row 0
    size_t rows_alloc = 0;
    float *x = nullptr, *y = nullptr, *h32 = nullptr, *pre = nullptr, *q32 = nullptr, *gate = nullptr, *logits_r = nullptr;
    void *h = nullptr, *mix = nullptr, *qt = nullptr;
    LatentScratch lat;
    void *k_exp = nullptr, *v_exp = nullptr;
    size_t exp_rows = 0;  // positions k_exp / v_exp hold
    uint32_t *ids = nullptr, *counts = nullptr, *cursor = nullptr, *entry_of = nullptr, *n_tiles = nullptr, *rows_dev = nullptr;
    MoeTile *tiles = nullptr;
    float *pick_w = nullptr, *col_scale = nullptr, *eo = nullptr;
    void *gathered = nullptr, *act = nullptr;
};

LayeredModel *as_layered(cera_cuda_model *m) { return dynamic_cast<LayeredModel *>(m); }

PadMap at(uint32_t base) {
    PadMap p;
    p.base = base;
    return p;
}
// groups of `group` entries padded to group_p, entries from `seg` on starting at seg_p, everything shifted by base
PadMap heads_map(uint32_t group, uint32_t group_p, uint32_t base = 0, uint32_t seg = 0xFFFFFFFFu, uint32_t seg_p = 0) {
    return PadMap{group, group_p, seg, seg_p, base};
}

int32_t LayeredModel::dense(DenseView *v, uint32_t rows, uint32_t cols_p, int as_f32) {
    v->rows = rows;
    v->ld = cols_p;
    v->f32 = as_f32;
    void *p = nullptr;
    const size_t bytes = (size_t)rows * cols_p * (as_f32 ? 4 : 2);
    CERA_TRY(dev_alloc(&p, bytes));
    v->w = p;
    return check_cuda(cudaMemset(p, 0, bytes), "cudaMemset(dense weight)");
}

int32_t LayeredModel::vec(float **p, uint32_t n) {
    CERA_TRY(dev_alloc((void **)p, (size_t)n * 4));
    return check_cuda(cudaMemset(*p, 0, (size_t)n * 4), "cudaMemset(vector)");
}

int32_t LayeredModel::place_layers() {
    CERA_TRY(dense(&embd, cfg.vocab_size, ld, f32));
    CERA_TRY(dense(&head, cfg.vocab_size, ld, f32));
    if (cfg.bigram_buckets) CERA_TRY(dense(&bigram, cfg.bigram_buckets + 1, ld, f32));
    for (auto &L : layers) {
        const auto &d = L.d;
        L.seen.assign(S_EXPERTS + 3 * (size_t)d.n_experts, false);
        if (d.mixer == CERA_MIXER_LATENT_ATTENTION) {
            has_attention = true;
            LatentShape &s = L.s;
            s.heads = d.n_heads;
            s.dim = d.head_dim;
            s.rot = d.rot_dim;
            s.vdim = d.value_dim;
            s.rank = d.kv_rank;
            s.dim_p = pad_to(s.dim, 16);
            s.rot_p = pad_to(s.rot, 16);
            s.vdim_p = pad_to(s.vdim, 16);
            s.rank_p = pad_to(s.rank, 64);
            s.in_p = pad_to(s.off_g() + s.heads, 4);
            s.scale = d.attn_scale;
            CERA_TRY(dense(&L.in, s.in_p, ld, f32));
            CERA_TRY(dense(&L.uk, s.heads * s.dim_p, s.rank_p, f32));
            CERA_TRY(dense(&L.uv, s.heads * s.vdim_p, s.rank_p, f32));
            CERA_TRY(dense(&L.out, ld, pad_to(s.heads * s.vdim_p, 64), f32));
            CERA_TRY(vec(&L.c_norm, s.rank_p));
            CERA_TRY(vec(&L.sink, s.heads));
        } else {
            has_recurrence = true;
            L.wp = pad_to(d.recurrent_width, 64);
            CERA_TRY(dense(&L.in, 3 * L.wp, ld, f32));
            CERA_TRY(dense(&L.out, ld, L.wp, f32));
            CERA_TRY(vec(&L.z_bias, L.wp));
            CERA_TRY(vec(&L.x_bias, L.wp));
            CERA_TRY(vec(&L.state, L.wp));
        }
        if (d.ff == CERA_FF_MOE) {
            L.ffn.ff_p = pad_to(d.ff_width, 64);
            CERA_TRY(dense(&L.ffn.gate_up, d.n_experts * 2 * L.ffn.ff_p, ld, f32));
            CERA_TRY(dense(&L.ffn.down, d.n_experts * ld, L.ffn.ff_p, f32));
            CERA_TRY(dense(&L.ffn.router, d.n_experts, ld, 1));
        }
    }
    return CERA_CUDA_OK;
}

// bytes (host or device) -> the padded place of a matrix, through a staging copy on the device
int32_t LayeredModel::place(const void *bytes, size_t nbytes, int32_t type, size_t rows, size_t cols, const DenseView &v, const PadMap &rmap,
                            const PadMap &cmap) {
    const size_t each = type == CERA_TYPE_F32 ? 4 : 2;
    if (type != CERA_TYPE_F32 && type != CERA_TYPE_F16 && type != CERA_TYPE_BF16)
        return fail(CERA_CUDA_ERR_UNSUPPORTED, "add_tensor: ggml type %d is not F32, F16 or BF16", type);
    if (nbytes != rows * cols * each) return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: %zu bytes for [%zu x %zu] of type %d", nbytes, rows, cols, type);
    void *raw = nullptr;
    CERA_CUDA_TRY(cudaMalloc(&raw, nbytes));
    int32_t rc = check_cuda(cudaMemcpy(raw, bytes, nbytes, cudaMemcpyDefault), "cudaMemcpy(weight)");
    if (rc == CERA_CUDA_OK) rc = launch_place(raw, type, rows, cols, const_cast<void *>(v.w), v.f32, v.ld, rmap, cmap, nullptr);
    if (rc == CERA_CUDA_OK) rc = check_cuda(cudaDeviceSynchronize(), "place");
    cudaFree(raw);
    return rc;
}

int32_t LayeredModel::add_tensor(int32_t role, int32_t layer, int32_t type, size_t rows, size_t cols, const void *bytes, size_t nbytes) {
    const bool global = role == CERA_ROLE_TOKEN_EMBD || role == CERA_ROLE_OUTPUT || role == CERA_ROLE_OUTPUT_NORM || role == CERA_ROLE_BIGRAM_EMBD;
    if (!global && (layer < 0 || (uint32_t)layer >= cfg.n_layers)) return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: layer %d out of range", layer);
    const uint32_t W = cfg.hidden_size;
    auto matrix = [&](const DenseView &v, size_t want_r, size_t want_c, const PadMap &rmap, const PadMap &cmap) -> int32_t {
        if (rows != want_r || cols != want_c || !v.w)
            return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: role %d layer %d expects [%zu x %zu], got [%zu x %zu]", role, layer, v.w ? want_r : 0, v.w ? want_c : 0, rows, cols);
        return place(bytes, nbytes, type, rows, cols, v, rmap, cmap);
    };
    auto vector = [&](float *p, size_t n) -> int32_t {
        if (rows * cols != n || !p) return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: role %d layer %d expects %zu numbers, got %zu", role, layer, p ? n : 0, rows * cols);
        DenseView v;
        v.w = p;
        v.rows = 1;
        v.ld = (uint32_t)n;
        v.f32 = 1;
        return place(bytes, nbytes, type, 1, n, v, at(0), at(0));
    };
    auto norm = [&](NormView *nv) -> int32_t {  // one number, or one per channel
        const size_t n = rows * cols;
        if (n != 1 && n != W) return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: norm of role %d layer %d has %zu numbers", role, layer, n);
        float *p = nullptr;
        CERA_TRY(vec(&p, n > 1 ? ld : 1));
        nv->g = p;
        nv->per_channel = n > 1 || W == 1;
        return vector(p, n);
    };
    switch (role) {
        case CERA_ROLE_TOKEN_EMBD: embd_seen = true; return matrix(embd, cfg.vocab_size, W, at(0), at(0));
        case CERA_ROLE_OUTPUT: head_seen = true; return matrix(head, cfg.vocab_size, W, at(0), at(0));
        case CERA_ROLE_BIGRAM_EMBD: bigram_seen = true; return matrix(bigram, (size_t)cfg.bigram_buckets + 1, W, at(0), at(0));
        case CERA_ROLE_OUTPUT_NORM: return norm(&out_norm);
        default: break;
    }
    LayerState &L = layers[layer];
    const auto &d = L.d;
    const LatentShape &s = L.s;
    const bool latent = d.mixer == CERA_MIXER_LATENT_ATTENTION;
    int slot = -1;
    auto take = [&](int sl, bool fits) {
        if (!fits) return false;
        slot = sl;
        return true;
    };
    const int32_t wrong = CERA_CUDA_ERR_BAD_ARG;
    auto misfit = [&] { return fail(wrong, "add_tensor: role %d does not belong to layer %d", role, layer); };
    auto done = [&](int32_t rc) {
        if (rc == CERA_CUDA_OK) L.seen[slot] = true;
        return rc;
    };
    switch (role) {
        case CERA_ROLE_MIX_PRE_NORM: slot = S_PRE; return done(norm(&L.pre));
        case CERA_ROLE_MIX_POST_NORM: slot = S_POST; return done(norm(&L.post));
        case CERA_ROLE_FF_PRE_NORM: return take(S_FF_PRE, d.ff != CERA_FF_NONE) ? done(norm(&L.ff_pre)) : misfit();
        case CERA_ROLE_FF_POST_NORM: return take(S_FF_POST, d.ff != CERA_FF_NONE) ? done(norm(&L.ff_post)) : misfit();
        case CERA_ROLE_MIX_OUTPUT:
            slot = S_OUT;
            return done(latent ? matrix(L.out, W, (size_t)s.heads * s.vdim, at(0), heads_map(s.vdim, s.vdim_p)) : matrix(L.out, W, d.recurrent_width, at(0), at(0)));
        case CERA_ROLE_LATENT_Q:
            if (!take(S_A, latent)) return misfit();
            return done(matrix(L.in, (size_t)s.heads * (s.dim + s.rot), W, heads_map(s.dim + s.rot, s.dim_p + s.rot_p, 0, s.dim, s.dim_p), at(0)));
        case CERA_ROLE_LATENT_DOWN:
            if (!take(S_B, latent)) return misfit();
            return done(matrix(L.in, (size_t)s.rank + s.rot, W, heads_map(s.rank + s.rot, s.rank_p + s.rot_p, s.off_c(), s.rank, s.rank_p), at(0)));
        case CERA_ROLE_LATENT_NORM: return take(S_C, latent) ? done(vector(L.c_norm, s.rank)) : misfit();
        case CERA_ROLE_LATENT_UP_K: return take(S_D, latent) ? done(matrix(L.uk, (size_t)s.heads * s.dim, s.rank, heads_map(s.dim, s.dim_p), at(0))) : misfit();
        case CERA_ROLE_LATENT_UP_V: return take(S_E, latent) ? done(matrix(L.uv, (size_t)s.heads * s.vdim, s.rank, heads_map(s.vdim, s.vdim_p), at(0))) : misfit();
        case CERA_ROLE_LATENT_SINK: return take(S_F, latent) ? done(vector(L.sink, s.heads)) : misfit();
        case CERA_ROLE_LATENT_GATE: return take(S_G, latent) ? done(matrix(L.in, s.heads, W, at(s.off_g()), at(0))) : misfit();
        case CERA_ROLE_GRU_Z: return take(S_A, !latent) ? done(matrix(L.in, d.recurrent_width, W, at(0), at(0))) : misfit();
        case CERA_ROLE_GRU_X: return take(S_B, !latent) ? done(matrix(L.in, d.recurrent_width, W, at(L.wp), at(0))) : misfit();
        case CERA_ROLE_GRU_GATE: return take(S_C, !latent) ? done(matrix(L.in, d.recurrent_width, W, at(2 * L.wp), at(0))) : misfit();
        case CERA_ROLE_GRU_Z_BIAS: return take(S_D, !latent) ? done(vector(L.z_bias, d.recurrent_width)) : misfit();
        case CERA_ROLE_GRU_X_BIAS: return take(S_E, !latent) ? done(vector(L.x_bias, d.recurrent_width)) : misfit();
        case CERA_ROLE_ROUTER: return take(S_ROUTER, d.ff == CERA_FF_MOE) ? done(matrix(L.ffn.router, d.n_experts, W, at(0), at(0))) : misfit();
        default: return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: unknown role %d for layer %d", role, layer);
    }
}

int32_t LayeredModel::add_expert(int32_t role, uint32_t layer, uint32_t expert, int32_t type, size_t rows, size_t cols, const void *bytes, size_t nbytes) {
    if (layer >= cfg.n_layers || layers[layer].d.ff != CERA_FF_MOE || expert >= layers[layer].d.n_experts)
        return fail(CERA_CUDA_ERR_BAD_ARG, "add_expert_tensor: layer %u has no expert %u", layer, expert);
    if (role < CERA_ROLE_EXPERT_GATE || role > CERA_ROLE_EXPERT_DOWN) return fail(CERA_CUDA_ERR_BAD_ARG, "add_expert_tensor: role %d", role);
    LayerState &L = layers[layer];
    const uint32_t W = cfg.hidden_size, ff = L.d.ff_width, ff_p = L.ffn.ff_p;
    const bool down = role == CERA_ROLE_EXPERT_DOWN;
    if (rows != (down ? W : ff) || cols != (down ? ff : W))
        return fail(CERA_CUDA_ERR_BAD_ARG, "add_expert_tensor: role %d expects [%u x %u], got [%zu x %zu]", role, down ? W : ff, down ? ff : W, rows, cols);
    // the base row may exceed 32 bits times the row length, not 32 bits
    const PadMap rmap = at(down ? expert * ld : expert * 2 * ff_p + (role == CERA_ROLE_EXPERT_UP ? ff_p : 0));
    CERA_TRY(place(bytes, nbytes, type, rows, cols, down ? L.ffn.down : L.ffn.gate_up, rmap, at(0)));
    L.seen[S_EXPERTS + 3 * (size_t)expert + (role - CERA_ROLE_EXPERT_GATE)] = true;
    return CERA_CUDA_OK;
}

int32_t LayeredModel::build() {
    if (!embd_seen || !head_seen || !out_norm.g || (cfg.bigram_buckets && !bigram_seen))
        return fail(CERA_CUDA_ERR_STATE, "finalize: an embedding, the head or the final norm is missing");
    for (uint32_t i = 0; i < cfg.n_layers; ++i) {
        const LayerState &L = layers[i];
        const bool latent = L.d.mixer == CERA_MIXER_LATENT_ATTENTION, moe = L.d.ff == CERA_FF_MOE;
        for (size_t sl = 0; sl < L.seen.size(); ++sl) {
            const bool need = sl == S_PRE || sl == S_POST || sl == S_OUT || (sl >= S_A && sl <= S_E) || ((sl == S_F || sl == S_G) && latent) ||
                              ((sl == S_FF_PRE || sl == S_FF_POST || sl >= S_ROUTER) && moe);
            if (need && !L.seen[sl]) return fail(CERA_CUDA_ERR_STATE, "finalize: layer %u is missing a tensor (slot %zu)", i, sl);
        }
    }
    const size_t C = LAYERED_CHUNK < max_seq_len ? LAYERED_CHUNK : max_seq_len;
    size_t pre_w = 0, mix_w = 64, q_w = 0, ql = 0, part = 0, heads = 1, gather_w = 0, eo_rows = 0, ff_w = 0, experts = 1, used = 1, kx = 0, vx = 0;
    auto up = [](size_t &a, size_t b) { a = a > b ? a : b; };
    for (auto &L : layers) {
        up(pre_w, L.in.rows);
        up(mix_w, L.out.ld);
        if (L.d.mixer == CERA_MIXER_LATENT_ATTENTION) {
            const LatentShape &s = L.s;
            up(q_w, s.q_ld());
            up(heads, s.heads);
            up(ql, (size_t)s.heads * (s.rank_p + s.rot_p));
            up(part, (size_t)s.heads * (s.rank_p + 2));
            up(kx, (size_t)s.heads * s.dim_p);
            up(vx, (size_t)s.heads * s.vdim_p);
            CERA_TRY(dev_alloc(&L.cache_c, (size_t)max_seq_len * s.rank_p * esz));
            CERA_TRY(dev_alloc(&L.cache_r, (size_t)max_seq_len * s.rot_p * esz));
            // angle = position * base^(-2i / rot): the frequency and the angle in f32, cos / sin from the C library
            std::vector<float> t((size_t)max_seq_len * s.rot);
            for (uint32_t i = 0; i < s.rot / 2; ++i) {
                const float f = (float)std::pow((double)L.d.rope_base, -2.0 * i / s.rot);
                for (size_t p = 0; p < max_seq_len; ++p) {
                    const float a = (float)p * f;
                    t[p * s.rot + 2 * i] = (float)std::cos((double)a);
                    t[p * s.rot + 2 * i + 1] = (float)std::sin((double)a);
                }
            }
            CERA_TRY(dev_alloc((void **)&L.rope, t.size() * 4));
            CERA_CUDA_TRY(cudaMemcpy(L.rope, t.data(), t.size() * 4, cudaMemcpyHostToDevice));
        }
        if (L.d.ff == CERA_FF_MOE) {
            up(ff_w, L.ffn.ff_p);
            up(experts, L.d.n_experts);
            up(used, L.d.n_used);
            gather_w = ld;
            eo_rows = C * used;
        }
    }
    CERA_TRY(dev_alloc((void **)&final_hidden, (size_t)ld * 4));
    CERA_TRY(dev_alloc((void **)&x, C * ld * 4));
    CERA_TRY(dev_alloc((void **)&y, C * ld * 4));
    CERA_TRY(dev_alloc((void **)&h32, C * ld * 4));
    CERA_TRY(dev_alloc(&h, C * ld * esz));
    CERA_TRY(dev_alloc((void **)&pre, C * pre_w * 4));
    CERA_TRY(dev_alloc(&mix, C * mix_w * esz));  // padding columns meet zero weights: finite is enough
    CERA_CUDA_TRY(cudaMemset(mix, 0, C * mix_w * esz));
    CERA_TRY(dev_alloc((void **)&rows_dev, C * 4));
    if (has_attention) {
        CERA_TRY(dev_alloc((void **)&q32, C * q_w * 4));
        if (!f32) CERA_TRY(dev_alloc(&qt, C * q_w * esz));
        CERA_TRY(dev_alloc((void **)&gate, C * heads * 4));
        CERA_TRY(dev_alloc((void **)&lat.q_lat, LATENT_MAX_SPLITS * ql * 4));
        CERA_TRY(dev_alloc((void **)&lat.part, LATENT_MAX_SPLITS * part * 4));
        bool fast = false;
        for (auto &L : layers) fast |= !f32 && L.d.mixer == CERA_MIXER_LATENT_ATTENTION && latent_prefill_supports(L.s);
        if (fast) {
            exp_rows = pad_to(max_seq_len, 64);
            CERA_TRY(dev_alloc(&k_exp, exp_rows * kx * esz));
            CERA_TRY(dev_alloc(&v_exp, exp_rows * vx * esz));
            // positions never written are multiplied by a zero weight: they must not hold a NaN
            CERA_CUDA_TRY(cudaMemset(v_exp, 0, exp_rows * vx * esz));
        }
    }
    if (eo_rows) {
        eo_rows = C * used;
        CERA_TRY(dev_alloc((void **)&logits_r, experts * 4));
        CERA_TRY(dev_alloc((void **)&ids, eo_rows * 4));
        CERA_TRY(dev_alloc((void **)&pick_w, eo_rows * 4));
        CERA_TRY(dev_alloc((void **)&col_scale, eo_rows * 4));
        CERA_TRY(dev_alloc((void **)&entry_of, eo_rows * 4));
        CERA_TRY(dev_alloc((void **)&counts, experts * 4));
        CERA_CUDA_TRY(cudaMemset(counts, 0, experts * 4));
        CERA_TRY(dev_alloc((void **)&cursor, experts * 4));
        CERA_TRY(dev_alloc((void **)&n_tiles, 8));
        CERA_TRY(dev_alloc((void **)&tiles, (eo_rows / DENSE_GROUP_MIN + experts) * sizeof(MoeTile)));
        CERA_TRY(dev_alloc(&gathered, eo_rows * gather_w * esz));
        CERA_TRY(dev_alloc(&act, eo_rows * ff_w * esz));
        CERA_TRY(dev_alloc((void **)&eo, eo_rows * ld * 4));
    }
    rows_alloc = C;
    return CERA_CUDA_OK;
}

int32_t LayeredModel::enqueue_step(int kind, uint32_t splits) {
    cudaStream_t st = stream;
    CERA_TRY(launch_embed_dense(embd, bigram, bigram_rule, nullptr, dyn, 1, x, st));
    ResidualNorm rn;  // the boundary ahead of the next sublayer
    rn.x = x;
    rn.h = h;
    rn.h_f32 = f32;
    for (auto &L : layers) {
        rn.pre = L.pre;
        CERA_TRY(launch_residual_norm(rn, hidden_size, ld, 1, cfg.norm_eps, st));
        if (L.d.mixer == CERA_MIXER_MINGRU) {
            CERA_TRY(launch_mingru_step(L.in, h, L.z_bias, L.x_bias, L.state, mix, st));
        } else {
            CERA_TRY(launch_dense_gemv(L.in, h, pre, st));
            CERA_TRY(launch_latent_prepare(pre, L.s, 1, 0, dyn + DYN_POS, L.c_norm, cfg.norm_eps, L.rope, L.cache_c, L.cache_r, f32, q32, nullptr, gate, st));
            CERA_TRY(launch_latent_attention(q32, L.s, L.uk, L.uv, L.cache_c, L.cache_r, L.sink, gate, 1, 0, dyn + DYN_LEN, splits, lat, mix, L.out.ld, st));
        }
        CERA_TRY(launch_dense_gemv(L.out, mix, y, st));
        rn.y = y;
        rn.post = L.post;
        if (L.d.ff == CERA_FF_MOE) {
            const RouterRule rule{L.d.n_experts, L.d.n_used, L.d.router_softmax, L.d.router_renorm, L.d.weight_input};
            const ExpertAct ea{L.d.act_limit, L.d.act_alpha, L.d.act_shift};
            rn.pre = L.ff_pre;
            rn.h32 = h32;
            CERA_TRY(launch_residual_norm(rn, hidden_size, ld, 1, cfg.norm_eps, st));
            rn.h32 = nullptr;
            CERA_TRY(launch_dense_gemv(L.ffn.router, h32, logits_r, st));
            CERA_TRY(launch_expert_gate_up_step(L.ffn.gate_up, h, logits_r, rule, L.ffn.ff_p, ea, ids, pick_w, act, st));
            CERA_TRY(launch_expert_down_step(L.ffn.down, ld, act, rule, ids, pick_w, y, st));
            rn.post = L.ff_post;
        }
    }
    if (kind == G_BODY) return CERA_CUDA_OK;  // the state has moved on; nothing reads the last boundary
    rn.pre = out_norm;
    rn.h32 = final_hidden;
    CERA_TRY(launch_residual_norm(rn, hidden_size, ld, 1, cfg.norm_eps, st));
    CERA_TRY(launch_dense_gemv(head, h, logits, st));
    if (kind == G_GREEDY || kind == G_CHAIN) CERA_TRY(launch_argmax(logits, vocab_size, tok_out, argmax_scratch, st));
    return kind == G_CHAIN ? launch_advance() : CERA_CUDA_OK;
}

// The mixer over a chunk: h -> `mix` -> y.
int32_t LayeredModel::mixer_chunk(LayerState &L, size_t n, size_t start_pos, float *y_out) {
    DenseGemm g;
    g.w = L.in;
    g.x = h;
    g.n = (uint32_t)n;
    g.out = pre;
    g.ldo = L.in.rows;
    CERA_TRY(launch_dense_gemm(g, stream));
    if (L.d.mixer == CERA_MIXER_MINGRU) CERA_TRY(launch_mingru_scan(pre, n, L.wp, L.z_bias, L.x_bias, L.state, mix, f32, stream));
    else CERA_TRY(latent_chunk(L, n, start_pos));
    DenseGemm o;
    o.w = L.out;
    o.x = mix;
    o.n = (uint32_t)n;
    o.out = y_out;
    o.ldo = ld;
    return launch_dense_gemm(o, stream);
}

int32_t LayeredModel::latent_chunk(LayerState &L, size_t n, size_t start_pos) {
    const LatentShape &s = L.s;
    const size_t ldm = L.out.ld;
    const bool expand = !f32 && n >= LATENT_EXPAND_MIN && k_exp && latent_prefill_supports(s);
    CERA_TRY(launch_latent_prepare(pre, s, n, start_pos, nullptr, L.c_norm, cfg.norm_eps, L.rope, L.cache_c, L.cache_r, f32, expand ? nullptr : q32,
                                   expand ? qt : nullptr, gate, stream));
    if (expand) {
        DenseGemm k;
        k.w = L.uk;
        k.x = L.cache_c;
        k.n = (uint32_t)(start_pos + n);
        k.out_kind = DENSE_T;
        k.out = k_exp;
        k.ldo = (size_t)s.heads * s.dim_p;
        CERA_TRY(launch_dense_gemm(k, stream));
        DenseGemm v = k;
        v.w = L.uv;
        v.out_kind = DENSE_T_TRANSPOSED;
        v.out = v_exp;
        v.ldo = exp_rows;
        CERA_TRY(launch_dense_gemm(v, stream));
        bool taken = false;
        CERA_TRY(launch_latent_prefill(qt, s, k_exp, L.cache_r, max_seq_len, v_exp, exp_rows, L.sink, gate, n, start_pos, mix, ldm, stream, &taken));
        return taken ? CERA_CUDA_OK : fail(CERA_CUDA_ERR_STATE, "latent attention: no kernel for the expanded form");
    }
    uint32_t splits = latent_splits(start_pos + n);
    size_t cn = 0;
    for (size_t j = 0; j < n; j += cn) {
        cn = n - j < LATENT_MAX_SPLITS ? n - j : LATENT_MAX_SPLITS;
        uint32_t sp = splits;
        while (sp > 1 && cn * sp > LATENT_MAX_SPLITS) sp /= 2;
        CERA_TRY(launch_latent_attention(q32 + j * s.q_ld(), s, L.uk, L.uv, L.cache_c, L.cache_r, L.sink, gate + j * s.heads, cn, start_pos + j, nullptr, sp,
                                         lat, (char *)mix + j * ldm * esz, ldm, stream));
    }
    return CERA_CUDA_OK;
}

// The routed feed-forward over a chunk: h, h32 -> `eo` in bucket order; `next` sums the picks.
int32_t LayeredModel::experts_chunk(LayerState &L, size_t n, ResidualNorm *next) {
    const auto &d = L.d;
    const uint32_t entries = (uint32_t)(n * d.n_used), columns = dense_group_columns(entries, d.n_experts), max_tiles = entries / columns + d.n_experts;
    CERA_TRY(launch_moe_route(h32, ld, n, (const float *)L.ffn.router.w, nullptr, ld, d.n_experts, d.n_used, d.router_softmax, d.router_renorm, ids, pick_w,
                              counts, stream));
    CERA_TRY(launch_moe_plan(counts, d.n_experts, columns, 0, 0, cursor, tiles, n_tiles, stream));
    CERA_TRY(launch_moe_gather(h, f32, ld, ids, pick_w, d.n_used, n, cursor, entry_of, gathered, col_scale, stream));
    DenseGemm g;
    g.w = L.ffn.gate_up;
    g.x = gathered;
    g.n = entries;
    g.out_kind = DENSE_GATED_UNIT;
    g.out = act;
    g.ldo = L.ffn.ff_p;
    g.tiles = tiles;
    g.n_tiles = n_tiles;
    g.max_tiles = max_tiles;
    g.rows_per_expert = 2 * L.ffn.ff_p;
    g.group_columns = columns;
    g.act = ExpertAct{d.act_limit, d.act_alpha, d.act_shift};
    g.col_scale = d.weight_input ? col_scale : nullptr;
    CERA_TRY(launch_dense_gemm(g, stream));
    DenseGemm o;
    o.w = L.ffn.down;
    o.x = act;
    o.n = entries;
    o.out = eo;
    o.ldo = ld;
    o.tiles = tiles;
    o.n_tiles = n_tiles;
    o.max_tiles = max_tiles;
    o.rows_per_expert = ld;
    o.group_columns = columns;
    CERA_TRY(launch_dense_gemm(o, stream));
    next->y = eo;
    next->entry_of = entry_of;
    next->picks = d.n_used;
    next->pick_weight = d.weight_input ? nullptr : pick_w;
    next->post = L.ff_post;
    return CERA_CUDA_OK;
}

int32_t LayeredModel::prefill_chunk(const uint32_t *tokens, size_t n, size_t start_pos) {
    cudaStream_t st = stream;
    const uint64_t before = launches_so_far();
    std::vector<uint32_t> t(n + 1);
    t[0] = token_before(start_pos);
    memcpy(t.data() + 1, tokens, n * 4);
    CERA_CUDA_TRY(cudaMemcpyAsync(pf_tokens, t.data(), (n + 1) * 4, cudaMemcpyHostToDevice, st));
    CERA_TRY(launch_embed_dense(embd, bigram, bigram_rule, pf_tokens, nullptr, n, x, st));
    ResidualNorm rn;
    rn.x = x;
    rn.h = h;
    rn.h_f32 = f32;
    for (auto &L : layers) {
        rn.pre = L.pre;
        CERA_TRY(launch_residual_norm(rn, hidden_size, ld, n, cfg.norm_eps, st));
        CERA_TRY(mixer_chunk(L, n, start_pos, y));
        rn.y = y;
        rn.entry_of = nullptr;
        rn.post = L.post;
        if (L.d.ff == CERA_FF_MOE) {
            rn.pre = L.ff_pre;
            rn.h32 = h32;
            CERA_TRY(launch_residual_norm(rn, hidden_size, ld, n, cfg.norm_eps, st));
            rn.h32 = nullptr;
            CERA_TRY(experts_chunk(L, n, &rn));
        }
    }
    rn.pre = out_norm;  // completes x; the head norms the rows it is asked for
    rn.h32 = nullptr;
    CERA_TRY(launch_residual_norm(rn, hidden_size, ld, n, cfg.norm_eps, st));
    launches += launches_so_far() - before;
    return CERA_CUDA_OK;
}

int32_t LayeredModel::logits_of_last(size_t n) {
    const uint64_t before = launches_so_far();
    ResidualNorm rn;
    rn.x = x + (n - 1) * ld;
    rn.pre = out_norm;
    rn.h = h;
    rn.h_f32 = f32;
    rn.h32 = final_hidden;
    CERA_TRY(launch_residual_norm(rn, hidden_size, ld, 1, cfg.norm_eps, stream));
    CERA_TRY(launch_dense_gemv(head, h, logits, stream));
    launches += launches_so_far() - before;
    return CERA_CUDA_OK;
}

int32_t LayeredModel::logits_of_rows(const uint32_t *rows, size_t n_rows, size_t n, float *out) {
    const uint64_t before = launches_so_far();
    constexpr size_t STEP = 256;  // rows of logits held on the device at a time
    if (!pf_logits) CERA_TRY(dev_alloc((void **)&pf_logits, STEP * (size_t)vocab_size * 4));
    if (rows) CERA_CUDA_TRY(cudaMemcpyAsync(rows_dev, rows, n_rows * 4, cudaMemcpyHostToDevice, stream));
    else n_rows = n;
    size_t cn = 0;
    for (size_t i = 0; i < n_rows; i += cn) {
        cn = n_rows - i < STEP ? n_rows - i : STEP;
        ResidualNorm rn;
        rn.x = rows ? x : x + i * ld;
        rn.x_rows = rows ? rows_dev + i : nullptr;
        rn.pre = out_norm;
        rn.h = h;
        rn.h_f32 = f32;
        CERA_TRY(launch_residual_norm(rn, hidden_size, ld, cn, cfg.norm_eps, stream));
        DenseGemm g;
        g.w = head;
        g.x = h;
        g.n = (uint32_t)cn;
        g.out = pf_logits;
        g.ldo = vocab_size;
        CERA_TRY(launch_dense_gemm(g, stream));
        CERA_CUDA_TRY(cudaMemcpyAsync(out + i * vocab_size, pf_logits, cn * vocab_size * 4, cudaMemcpyDeviceToHost, stream));
    }
    launches += launches_so_far() - before;
    return CERA_CUDA_OK;
}

int32_t LayeredModel::rewind(size_t len) {
    // latents beyond len are overwritten later; a recurrent state exists for the current position only
    if (len && has_recurrence)
        return fail(CERA_CUDA_ERR_UNSUPPORTED, "truncate_kv: recurrent layers keep no state of position %zu (restore a snapshot, or truncate to 0)", len);
    if (!finalized) return CERA_CUDA_OK;
    if (len == 0)
        for (auto &L : layers)
            if (L.state) CERA_CUDA_TRY(cudaMemsetAsync(L.state, 0, (size_t)L.wp * 4, stream));
    return check_cuda(cudaStreamSynchronize(stream), "truncate_kv");
}

struct LayeredSnapshot {
    uint32_t magic, version, n_layers, elem_bytes;
    uint64_t seq_len, bytes;
};
constexpr uint32_t LAYERED_MAGIC = 0x4C4B4243u;  // "CBKL"

// header, the consumed tokens, then per layer the latents and rotated parts of every position, or the state
size_t LayeredModel::snapshot_bytes() const {
    size_t n = sizeof(LayeredSnapshot) + seq_len * 4;
    for (const auto &L : layers) n += L.state ? (size_t)L.wp * 4 : seq_len * (L.s.rank_p + L.s.rot_p) * esz;
    return n;
}

int32_t LayeredModel::snapshot(void *out, size_t out_bytes) {
    const size_t need = snapshot_bytes();
    if (out_bytes < need) return fail(CERA_CUDA_ERR_BAD_ARG, "kv_snapshot: %zu bytes given, %zu needed", out_bytes, need);
    CERA_CUDA_TRY(cudaStreamSynchronize(stream));
    const LayeredSnapshot hd{LAYERED_MAGIC, 1, cfg.n_layers, (uint32_t)esz, (uint64_t)seq_len, (uint64_t)need};
    memcpy(out, &hd, sizeof(hd));
    char *p = (char *)out + sizeof(hd);
    memcpy(p, history.data(), seq_len * 4);
    p += seq_len * 4;
    auto get = [&](const void *src, size_t n) {
        const int32_t rc = n ? check_cuda(cudaMemcpy(p, src, n, cudaMemcpyDeviceToHost), "cudaMemcpy(snapshot)") : CERA_CUDA_OK;
        p += n;
        return rc;
    };
    for (auto &L : layers) {
        if (L.state) {
            CERA_TRY(get(L.state, (size_t)L.wp * 4));
        } else {
            CERA_TRY(get(L.cache_c, seq_len * L.s.rank_p * esz));
            CERA_TRY(get(L.cache_r, seq_len * L.s.rot_p * esz));
        }
    }
    return CERA_CUDA_OK;
}

int32_t LayeredModel::restore(const void *data, size_t bytes) {
    LayeredSnapshot hd;
    if (bytes < sizeof(hd)) return fail(CERA_CUDA_ERR_BAD_ARG, "kv_restore: %zu bytes is shorter than the header", bytes);
    memcpy(&hd, data, sizeof(hd));
    if (hd.magic != LAYERED_MAGIC || hd.version != 1 || hd.n_layers != cfg.n_layers || hd.elem_bytes != esz)
        return fail(CERA_CUDA_ERR_BAD_ARG, "kv_restore: not a snapshot of this model");
    if (hd.seq_len > max_seq_len) return fail(CERA_CUDA_ERR_BAD_ARG, "kv_restore: %llu positions exceed max_seq_len %u", (unsigned long long)hd.seq_len, max_seq_len);
    const size_t n = (size_t)hd.seq_len;
    size_t need = sizeof(hd) + n * 4;
    for (const auto &L : layers) need += L.state ? (size_t)L.wp * 4 : n * (L.s.rank_p + L.s.rot_p) * esz;
    if (bytes != need || hd.bytes != need) return fail(CERA_CUDA_ERR_BAD_ARG, "kv_restore: %zu bytes, %zu expected", bytes, need);
    CERA_CUDA_TRY(cudaStreamSynchronize(stream));
    const char *p = (const char *)data + sizeof(hd);
    history.assign((const uint32_t *)p, (const uint32_t *)p + n);
    p += n * 4;
    auto put = [&](void *dst, size_t b) {
        const int32_t rc = b ? check_cuda(cudaMemcpy(dst, p, b, cudaMemcpyHostToDevice), "cudaMemcpy(restore)") : CERA_CUDA_OK;
        p += b;
        return rc;
    };
    for (auto &L : layers) {
        if (L.state) {
            CERA_TRY(put(L.state, (size_t)L.wp * 4));
        } else {
            CERA_TRY(put(L.cache_c, n * L.s.rank_p * esz));
            CERA_TRY(put(L.cache_r, n * L.s.rot_p * esz));
        }
    }
    seq_len = n;
    return CERA_CUDA_OK;
}

int32_t check_layer(uint32_t i, const cera_cuda_layer_desc &d) {
    if (d.mixer == CERA_MIXER_LATENT_ATTENTION) {
        if (!d.n_heads || !d.head_dim || !d.rot_dim || d.rot_dim % 2 || !d.value_dim || !d.kv_rank || !(d.rope_base > 0.0f))
            return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: layer %u: latent attention sizes", i);
        if (d.kv_rank > 1024 || d.n_heads > 1024) return fail(CERA_CUDA_ERR_UNSUPPORTED, "model_create: layer %u: rank %u (at most 1024), %u heads", i, d.kv_rank, d.n_heads);
    } else if (d.mixer == CERA_MIXER_MINGRU) {
        if (!d.recurrent_width) return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: layer %u: recurrent width is zero", i);
    } else {
        return fail(CERA_CUDA_ERR_UNSUPPORTED, "model_create: layer %u: unknown mixer %d", i, d.mixer);
    }
    if (d.ff == CERA_FF_NONE) return CERA_CUDA_OK;
    if (d.ff != CERA_FF_MOE) return fail(CERA_CUDA_ERR_UNSUPPORTED, "model_create: layer %u: unknown feed-forward %d", i, d.ff);
    if (!d.ff_width || !d.n_experts || d.n_experts > 256 || !d.n_used || d.n_used > 16 || d.n_used > d.n_experts)
        return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: layer %u: %u experts of width %u, %u used (at most 256 and 16)", i, d.n_experts, d.ff_width, d.n_used);
    return CERA_CUDA_OK;
}

}  // namespace

extern "C" {

int32_t cera_cuda_model_create_layered(const cera_cuda_layered_config *cfg, const cera_cuda_layer_desc *descs, cera_cuda_model **out) {
    if (!cfg || !descs || !out) return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: null argument");
    const auto &c = *cfg;
    if (!c.n_layers || !c.hidden_size || !c.vocab_size || !c.max_seq_len) return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: zero dimension in config");
    if (c.dtype != CERA_TYPE_BF16 && c.dtype != CERA_TYPE_F32) return fail(CERA_CUDA_ERR_UNSUPPORTED, "model_create: dtype %d is not BF16 or F32", c.dtype);
    for (uint32_t i = 0; i < c.n_layers; ++i) CERA_TRY(check_layer(i, descs[i]));
    int n_dev = 0;
    CERA_CUDA_TRY(cudaGetDeviceCount(&n_dev));
    if (c.device < 0 || c.device >= n_dev) return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: device %d of %d", c.device, n_dev);
    DeviceGuard dg(c.device);
    auto *m = new (std::nothrow) LayeredModel(c, descs);
    if (!m) return fail(CERA_CUDA_ERR_OOM, "model_create: host allocation failed");
    const int32_t rc = m->place_layers();
    if (rc != CERA_CUDA_OK) {
        delete m;
        return rc;
    }
    *out = m;
    return CERA_CUDA_OK;
}

int32_t cera_cuda_model_add_expert_tensor(cera_cuda_model *m, int32_t role, int32_t layer, int32_t expert, int32_t type, size_t rows, size_t cols,
                                          const void *bytes, size_t nbytes) {
    if (!m || !bytes) return fail(CERA_CUDA_ERR_BAD_ARG, "add_expert_tensor: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    LayeredModel *lm = as_layered(m);
    if (!lm) return fail(CERA_CUDA_ERR_UNSUPPORTED, "add_expert_tensor: not offered by this architecture");
    DeviceGuard dg(m->device);
    if (m->finalized) return fail(CERA_CUDA_ERR_STATE, "add_expert_tensor: model already finalized");
    return lm->add_expert(role, (uint32_t)layer, (uint32_t)expert, type, rows, cols, bytes, nbytes);
}

}  // extern "C"
