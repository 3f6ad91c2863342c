// A decoder described layer by layer: every layer names its token mixer (latent attention, minGRU, attention with grouped key /
// value heads, a real-gated linear recurrence, a state-space recurrence) and its feed-forward (routed experts, one gated
// unit, or none), weights are dense (bf16 or f32).  A sublayer is normed before and, in some designs, after:
// x += post(sublayer(pre(x))), and the boundary between two sublayers - the residual sum of one, the norm of the next -
// is one kernel.  A range of layers may run several times in a row: `runs` lists the layer runs, each with a state of its own.
//
// Per sequence a run holds: latent attention one latent and one rotated key part per position; grouped attention a key and a
// value per position and group; a recurrence its f32 state and, behind a short convolution, the convolution's last inputs.
// The bigram embedding needs the previous token (the base's history / dyn words).
//
// A decode step per layer: [boundary] -> minGRU: [z / candidate / gate products + state update] [output product];
// latent attention: [input products] [norm, rotation, cache append] [W_uk on the query] [split attention] [merge, W_uv, gate]
// [output product]; grouped attention: [input products] [bias, rotation, norm, cache append] [split attention] [merge] [output
// product]; real-gated recurrence: [input products] [convolution, gates, state, output gate] [output product]; state-space
// recurrence: [input products] [convolution, state] [gate, norm] [output product]; experts: [boundary] [router logits] [pick,
// gate / up, gated unit] [down, sum over picks]; one gated unit: [boundary] [gate / up, gated unit] [down].
// A prompt portion takes the same steps with many-column products, scans for the recurrences, and experts grouped by a
// device-built work list.
#include <cmath>
#include <cstring>
#include <new>
#include <vector>

#include "dense.h"
#include "model.h"

using namespace cera;

namespace {

constexpr size_t LAYERED_CHUNK = 2048;   // prompt tokens per chunk
constexpr size_t ATTENTION_TC_MIN = 16;  // shorter portions attend query by query

constexpr size_t SSM_CHUNK_MIN = 16;      // shorter portions are scanned token by token

struct ExpertFfn {
    DenseView gate_up, down, router;  // gate_up: per expert ff_p gate rows, ff_p up rows; router: f32
    uint32_t ff_p = 0;
};

struct LayerWeights {
    cera_cuda_layer_desc d{};
    NormView pre, post, ff_pre, ff_post;
    DenseView in, out;  // the mixer's input products stacked into one matrix; its output projection
    float *in_bias = nullptr;
    const float *rope = nullptr;
    // latent attention
    LatentShape s;
    DenseView uk, uv;
    float *c_norm = nullptr, *sink = nullptr;
    // grouped attention
    GroupedShape a;
    // minGRU
    uint32_t wp = 0;
    float *z_bias = nullptr, *x_bias = nullptr;
    // short convolution of a recurrence
    float *conv_w = nullptr, *conv_b = nullptr;
    // real-gated and state-space recurrences; their state pointers are a run's
    RglruView lru;
    float *gate_bias = nullptr, *lam = nullptr;
    SsmView ssm;
    float *dt_bias = nullptr, *a_log = nullptr, *skip = nullptr, *ssm_norm = nullptr;
    ExpertFfn ffn;
    std::vector<bool> seen;  // tensors given, by slot

    bool is(int32_t mixer) const { return d.mixer == mixer; }
    bool attends() const { return is(CERA_MIXER_LATENT_ATTENTION) || is(CERA_MIXER_ATTENTION); }
};

// One run of a layer, and what it keeps of a sequence.
struct LayerRun {
    uint32_t layer = 0;
    bool again = false;  // the first layer of a repeated pass: the embedding is added ahead of it
    void *cache_a = nullptr, *cache_b = nullptr;  // latents and rotated parts; keys [position] and values [value][position]
    float *state = nullptr, *ring = nullptr;
    size_t state_n = 0, ring_n = 0;
};

// S_A..: the mixer's own tensors in the order of mixer_slots(); S_EXPERTS..: gate, up, down of each expert, or of the one unit
enum Slot { S_PRE, S_POST, S_FF_PRE, S_FF_POST, S_OUT, S_A, S_B, S_C, S_D, S_E, S_F, S_G, S_H, S_I, S_J, S_K, S_ROUTER, S_EXPERTS };
int mixer_slots(const cera_cuda_layer_desc &d) {
    switch (d.mixer) {
        case CERA_MIXER_LATENT_ATTENTION: return 7;
        case CERA_MIXER_MINGRU: return 5;
        case CERA_MIXER_ATTENTION: return d.attn_bias ? 6 : 3;
        case CERA_MIXER_RGLRU: return 11;
        default: return 7;  // state-space
    }
}

struct LayeredModel : cera_cuda_model {
    LayeredModel(const cera_cuda_layered_config &c, const cera_cuda_layer_desc *l)
        : cera_cuda_model(c.vocab_size, c.hidden_size, c.max_seq_len, c.device), cfg(c), f32(c.dtype == CERA_TYPE_F32), esz(f32 ? 4 : 2),
          ld(pad_to(c.hidden_size, 64)), layers(c.n_layers) {
        for (uint32_t i = 0; i < c.n_layers; ++i) layers[i].d = l[i];
        bigram_rule.buckets = c.bigram_buckets;
        bigram_rule.mul_prev = c.bigram_mul_prev;
        bigram_rule.mul_cur = c.bigram_mul_cur;
        auto run = [&](uint32_t from, uint32_t to, bool again) {
            for (uint32_t i = from; i < to; ++i) {
                LayerRun r;
                r.layer = i;
                r.again = again && i == from;
                runs.push_back(r);
            }
        };
        const uint32_t times = c.loop_times > 1 ? c.loop_times : 1, stop = times > 1 ? c.loop_stop : c.n_layers;
        run(0, stop, false);
        for (uint32_t t = 1; t < times; ++t) run(c.loop_start, stop, true);
        run(stop, c.n_layers, false);
    }
    int32_t place_layers();  // allocates the weights and works out the padded shapes
    int32_t add_tensor(int32_t role, int32_t layer, int32_t type, size_t rows, size_t cols, const void *bytes, size_t nbytes) override;
    int32_t add_expert(int32_t role, uint32_t layer, uint32_t expert, int32_t type, size_t rows, size_t cols, const void *bytes, size_t nbytes);
    int32_t build() override;
    size_t chunk_tokens() const override { return LAYERED_CHUNK; }
    uint32_t plan(size_t n_positions) const override { return has_attention ? kv_splits(n_positions) : 1; }
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
    int32_t place(const void *bytes, size_t nbytes, int32_t type, size_t rows, size_t cols, const DenseView &v, const PadMap &rmap, const PadMap &cmap,
                  float offset = 0.0f);
    int32_t rope_table(float base, uint32_t rot, const float **out);
    int32_t mixer_chunk(LayerRun &R, size_t n, size_t start_pos, float *y);
    int32_t latent_chunk(LayerRun &R, size_t n, size_t start_pos);
    int32_t attention_chunk(LayerRun &R, size_t n, size_t start_pos);
    int32_t rglru_chunk(LayerRun &R, size_t n, size_t start_pos);
    int32_t ssm_chunk(LayerRun &R, size_t n, size_t start_pos);
    int32_t unit_chunk(LayerWeights &L, size_t n, ResidualNorm *next);
    float embedding_scale() const { return cfg.embedding_scale != 0.0f ? cfg.embedding_scale : 1.0f; }
    RglruView rglru_view(const LayerRun &R) const;
    SsmView ssm_view(const LayerRun &R) const;
    struct Piece {  // of a sequence's state: `rows` rows of `bytes`, `pitch` apart
        void *p;
        size_t bytes, rows, pitch;
    };
    std::vector<Piece> pieces(size_t n) const;  // of n positions, in the order of a snapshot
    int32_t experts_chunk(LayerWeights &L, size_t n, ResidualNorm *next);

    const cera_cuda_layered_config cfg;
    const int f32;
    const size_t esz;
    const uint32_t ld;
    BigramParams bigram_rule;
    bool has_attention = false, has_recurrence = false;
    DenseView embd, bigram, head;
    NormView out_norm;
    bool head_seen = false, embd_seen = false, bigram_seen = false;
    std::vector<LayerWeights> layers;
    std::vector<LayerRun> runs;
    size_t ld_v = 0;  // row length of the transposed value caches
    struct Rope {
        float base;
        uint32_t rot;
        float *table;
    };
    std::vector<Rope> ropes;
    // scratch; chunk buffers have LAYERED_CHUNK rows, the decode step uses row 0
    size_t rows_alloc = 0;
    float *x = nullptr, *emb = nullptr, *y = nullptr, *h32 = nullptr, *aux = nullptr, *pre = nullptr, *q32 = nullptr, *gate = nullptr, *logits_r = nullptr;
    void *h = nullptr, *mix = nullptr, *qt = nullptr, *conv = nullptr;
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
    if (!cfg.tied_output) CERA_TRY(dense(&head, cfg.vocab_size, ld, f32));
    if (cfg.bigram_buckets) CERA_TRY(dense(&bigram, cfg.bigram_buckets + 1, ld, f32));
    for (auto &L : layers) {
        const auto &d = L.d;
        L.seen.assign(S_EXPERTS + 3 * (size_t)(d.ff == CERA_FF_MOE ? d.n_experts : 1), false);
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
        } else if (d.mixer == CERA_MIXER_ATTENTION) {
            has_attention = true;
            GroupedShape &a = L.a;
            a.heads = d.n_heads;
            a.kv_heads = d.n_kv_heads;
            a.dim = d.head_dim;
            a.rot = d.rot_dim;
            a.vdim = d.value_dim;
            a.dim_p = pad_to(a.dim, 16);
            a.vdim_p = pad_to(a.vdim, 16);
            a.in_p = pad_to(a.in_rows(), 4);
            a.scale = d.attn_scale;
            a.softcap = d.softcap;
            a.eps = cfg.norm_eps;
            a.qk_norm = d.qk_norm;
            CERA_TRY(dense(&L.in, a.in_p, ld, f32));
            CERA_TRY(dense(&L.out, ld, pad_to(a.heads * a.vdim_p, 64), f32));
            CERA_TRY(vec(&L.in_bias, a.in_p));
        } else if (d.mixer == CERA_MIXER_RGLRU) {
            has_recurrence = true;
            RglruView &v = L.lru;
            v.block_p = pad_to(d.recurrent_width / d.n_blocks, 64);
            v.wp = d.n_blocks * v.block_p;
            v.decay = d.decay;
            CERA_TRY(dense(&L.in, 2 * v.wp, ld, f32));
            CERA_TRY(dense(&L.out, ld, v.wp, f32));
            CERA_TRY(dense(&v.gates, 2 * v.wp, v.block_p, f32));
            CERA_TRY(vec(&L.in_bias, 2 * v.wp));
            CERA_TRY(vec(&L.gate_bias, 2 * v.wp));
            CERA_TRY(vec(&L.lam, v.wp));
            CERA_TRY(vec(&L.conv_w, v.wp * d.conv_taps));
            CERA_TRY(vec(&L.conv_b, v.wp));
            v.in_bias = L.in_bias;
            v.gate_bias = L.gate_bias;
            v.lam = L.lam;
            v.conv = ConvView{L.conv_w, L.conv_b, nullptr, v.wp, d.conv_taps};
        } else if (d.mixer == CERA_MIXER_SSM) {
            has_recurrence = true;
            SsmShape &m = L.ssm.s;
            m.heads = d.n_heads;
            m.dim = d.value_dim;
            m.state = d.state_size;
            m.groups = d.n_groups;
            m.norm_groups = d.n_norm_groups;
            m.dim_p = pad_to(m.dim, 16);
            m.state_p = pad_to(m.state, 16);
            m.in_p = pad_to(m.in_rows(), 4);
            m.eps = cfg.norm_eps;
            CERA_TRY(dense(&L.in, m.in_p, ld, f32));
            CERA_TRY(dense(&L.out, ld, pad_to(m.inner_p(), 64), f32));
            CERA_TRY(vec(&L.conv_w, m.channels() * d.conv_taps));
            CERA_TRY(vec(&L.conv_b, m.channels()));
            CERA_TRY(vec(&L.dt_bias, m.heads));
            CERA_TRY(vec(&L.a_log, m.heads));
            CERA_TRY(vec(&L.skip, m.heads));
            CERA_TRY(vec(&L.ssm_norm, m.inner_p()));
            L.ssm.dt_bias = L.dt_bias;
            L.ssm.a_log = L.a_log;
            L.ssm.d = L.skip;
            L.ssm.norm = L.ssm_norm;
            L.ssm.conv = ConvView{L.conv_w, L.conv_b, nullptr, m.channels(), d.conv_taps};
        } else {
            has_recurrence = true;
            L.wp = pad_to(d.recurrent_width, 64);
            CERA_TRY(dense(&L.in, 3 * L.wp, ld, f32));
            CERA_TRY(dense(&L.out, ld, L.wp, f32));
            CERA_TRY(vec(&L.z_bias, L.wp));
            CERA_TRY(vec(&L.x_bias, L.wp));
        }
        if (d.ff == CERA_FF_MOE) {
            L.ffn.ff_p = pad_to(d.ff_width, 64);
            CERA_TRY(dense(&L.ffn.gate_up, d.n_experts * 2 * L.ffn.ff_p, ld, f32));
            CERA_TRY(dense(&L.ffn.down, d.n_experts * ld, L.ffn.ff_p, f32));
            CERA_TRY(dense(&L.ffn.router, d.n_experts, ld, 1));
        } else if (d.ff == CERA_FF_GATED) {
            L.ffn.ff_p = pad_to(d.ff_width, 64);
            CERA_TRY(dense(&L.ffn.gate_up, 2 * L.ffn.ff_p, ld, f32));
            CERA_TRY(dense(&L.ffn.down, ld, L.ffn.ff_p, f32));
        }
    }
    return CERA_CUDA_OK;
}

// bytes (host or device) -> the padded place of a matrix, through a staging copy on the device
int32_t LayeredModel::place(const void *bytes, size_t nbytes, int32_t type, size_t rows, size_t cols, const DenseView &v, const PadMap &rmap,
                            const PadMap &cmap, float offset) {
    const size_t each = type == CERA_TYPE_F32 ? 4 : 2;
    if (type != CERA_TYPE_F32 && type != CERA_TYPE_F16 && type != CERA_TYPE_BF16)
        return fail(CERA_CUDA_ERR_UNSUPPORTED, "add_tensor: ggml type %d is not F32, F16 or BF16", type);
    if (nbytes != rows * cols * each) return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: %zu bytes for [%zu x %zu] of type %d", nbytes, rows, cols, type);
    void *raw = nullptr;
    CERA_CUDA_TRY(cudaMalloc(&raw, nbytes));
    int32_t rc = check_cuda(cudaMemcpy(raw, bytes, nbytes, cudaMemcpyDefault), "cudaMemcpy(weight)");
    if (rc == CERA_CUDA_OK) rc = launch_place(raw, type, rows, cols, const_cast<void *>(v.w), v.f32, v.ld, rmap, cmap, nullptr, offset);
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
    // the tensor's rows in consecutive parts, each placed by a map of its own
    struct Part {
        size_t n;
        PadMap map;
    };
    auto parts = [&](const DenseView &v, std::initializer_list<Part> list) -> int32_t {
        size_t total = 0, at_row = 0;
        for (const Part &q : list) total += q.n;
        const size_t each = type == CERA_TYPE_F32 ? 4 : 2, c = rows * cols / (total ? total : 1);
        if (!v.w || rows * cols != total * c || (v.ld != ld && c != v.ld) || (v.ld == ld && c != W) || nbytes != total * c * each)
            return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: role %d layer %d: [%zu x %zu] is not %zu rows of the layer", role, layer, rows, cols, total);
        for (const Part &q : list) {
            CERA_TRY(place((const char *)bytes + at_row * c * each, q.n * c * each, type, q.n, c, v, q.map, at(0)));
            at_row += q.n;
        }
        return CERA_CUDA_OK;
    };
    // f32 rows of n numbers
    auto table = [](float *p, uint32_t n) {
        DenseView v;
        v.w = p;
        v.ld = n;
        v.f32 = 1;
        return v;
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
        DenseView v;
        v.w = p;
        v.rows = 1;
        v.ld = (uint32_t)n;
        v.f32 = 1;
        return place(bytes, nbytes, type, 1, n, v, at(0), at(0), cfg.norm_offset);
    };
    switch (role) {
        case CERA_ROLE_TOKEN_EMBD: embd_seen = true; return matrix(embd, cfg.vocab_size, W, at(0), at(0));
        case CERA_ROLE_OUTPUT:
            if (cfg.tied_output) return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: the output is the embedding");
            head_seen = true;
            return matrix(head, cfg.vocab_size, W, at(0), at(0));
        case CERA_ROLE_BIGRAM_EMBD: bigram_seen = true; return matrix(bigram, (size_t)cfg.bigram_buckets + 1, W, at(0), at(0));
        case CERA_ROLE_OUTPUT_NORM: return norm(&out_norm);
        default: break;
    }
    LayerWeights &L = layers[layer];
    const auto &d = L.d;
    const LatentShape &s = L.s;
    const GroupedShape &a = L.a;
    const SsmShape &m = L.ssm.s;
    const bool latent = L.is(CERA_MIXER_LATENT_ATTENTION), gru = L.is(CERA_MIXER_MINGRU), grouped = L.is(CERA_MIXER_ATTENTION), lru = L.is(CERA_MIXER_RGLRU),
               ssm = L.is(CERA_MIXER_SSM);
    const uint32_t block = lru ? d.recurrent_width / d.n_blocks : 0, wp = L.lru.wp, bp = L.lru.block_p;
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
        case CERA_ROLE_MIX_POST_NORM: return take(S_POST, !cfg.no_post_norms) ? done(norm(&L.post)) : misfit();
        case CERA_ROLE_FF_PRE_NORM: return take(S_FF_PRE, d.ff != CERA_FF_NONE) ? done(norm(&L.ff_pre)) : misfit();
        case CERA_ROLE_FF_POST_NORM: return take(S_FF_POST, d.ff != CERA_FF_NONE && !cfg.no_post_norms) ? done(norm(&L.ff_post)) : misfit();
        case CERA_ROLE_MIX_OUTPUT: {
            slot = S_OUT;
            if (latent) return done(matrix(L.out, W, (size_t)s.heads * s.vdim, at(0), heads_map(s.vdim, s.vdim_p)));
            if (grouped) return done(matrix(L.out, W, (size_t)a.heads * a.vdim, at(0), heads_map(a.vdim, a.vdim_p)));
            if (ssm) return done(matrix(L.out, W, (size_t)m.heads * m.dim, at(0), heads_map(m.dim, m.dim_p)));
            return done(matrix(L.out, W, d.recurrent_width, at(0), lru ? heads_map(block, bp) : at(0)));
        }
        case CERA_ROLE_ATTN_Q: return take(S_A, grouped) ? done(parts(L.in, {{(size_t)a.heads * a.dim, heads_map(a.dim, a.dim_p)}})) : misfit();
        case CERA_ROLE_ATTN_K: return take(S_B, grouped) ? done(parts(L.in, {{(size_t)a.kv_heads * a.dim, heads_map(a.dim, a.dim_p, a.off_k())}})) : misfit();
        case CERA_ROLE_ATTN_V: return take(S_C, grouped) ? done(parts(L.in, {{(size_t)a.kv_heads * a.vdim, heads_map(a.vdim, a.vdim_p, a.off_v())}})) : misfit();
        case CERA_ROLE_ATTN_Q_BIAS:
            if (!take(S_D, grouped && d.attn_bias)) return misfit();
            return done(parts(table(L.in_bias, 1), {{(size_t)a.heads * a.dim, heads_map(a.dim, a.dim_p)}}));
        case CERA_ROLE_ATTN_K_BIAS:
            if (!take(S_E, grouped && d.attn_bias)) return misfit();
            return done(parts(table(L.in_bias, 1), {{(size_t)a.kv_heads * a.dim, heads_map(a.dim, a.dim_p, a.off_k())}}));
        case CERA_ROLE_ATTN_V_BIAS:
            if (!take(S_F, grouped && d.attn_bias)) return misfit();
            return done(parts(table(L.in_bias, 1), {{(size_t)a.kv_heads * a.vdim, heads_map(a.vdim, a.vdim_p, a.off_v())}}));
        case CERA_ROLE_CONV:
        case CERA_ROLE_CONV_BIAS: {
            const bool w = role == CERA_ROLE_CONV;
            if (!take(ssm ? (w ? S_B : S_C) : w ? S_E : S_F, lru || ssm)) return misfit();
            const DenseView v = w ? table(L.conv_w, d.conv_taps) : table(L.conv_b, 1);
            const size_t inner = (size_t)m.heads * m.dim, gn = (size_t)m.groups * m.state;
            if (lru) return done(parts(v, {{d.recurrent_width, heads_map(block, bp)}}));
            return done(parts(v, {{inner, heads_map(m.dim, m.dim_p)}, {gn, heads_map(m.state, m.state_p, m.off_b())}, {gn, heads_map(m.state, m.state_p, m.off_c())}}));
        }
        case CERA_ROLE_LRU_OUT: return take(S_A, lru) ? done(parts(L.in, {{d.recurrent_width, heads_map(block, bp)}})) : misfit();
        case CERA_ROLE_LRU_OUT_BIAS: return take(S_B, lru) ? done(parts(table(L.in_bias, 1), {{d.recurrent_width, heads_map(block, bp)}})) : misfit();
        case CERA_ROLE_LRU_IN: return take(S_C, lru) ? done(parts(L.in, {{d.recurrent_width, heads_map(block, bp, wp)}})) : misfit();
        case CERA_ROLE_LRU_IN_BIAS: return take(S_D, lru) ? done(parts(table(L.in_bias, 1), {{d.recurrent_width, heads_map(block, bp, wp)}})) : misfit();
        case CERA_ROLE_LRU_DECAY_GATE: return take(S_G, lru) ? done(matrix(L.lru.gates, d.recurrent_width, block, heads_map(block, 2 * bp), at(0))) : misfit();
        case CERA_ROLE_LRU_DECAY_GATE_BIAS: return take(S_H, lru) ? done(parts(table(L.gate_bias, 1), {{d.recurrent_width, heads_map(block, 2 * bp)}})) : misfit();
        case CERA_ROLE_LRU_INPUT_GATE: return take(S_I, lru) ? done(matrix(L.lru.gates, d.recurrent_width, block, heads_map(block, 2 * bp, bp), at(0))) : misfit();
        case CERA_ROLE_LRU_INPUT_GATE_BIAS: return take(S_J, lru) ? done(parts(table(L.gate_bias, 1), {{d.recurrent_width, heads_map(block, 2 * bp, bp)}})) : misfit();
        case CERA_ROLE_LRU_LAMBDA: return take(S_K, lru) ? done(parts(table(L.lam, 1), {{d.recurrent_width, heads_map(block, bp)}})) : misfit();
        case CERA_ROLE_SSM_IN: {
            if (!take(S_A, ssm)) return misfit();
            const size_t inner = (size_t)m.heads * m.dim, gn = (size_t)m.groups * m.state;
            const uint32_t c0 = m.inner_p();  // the convolved channels follow z
            return done(parts(L.in, {{inner, heads_map(m.dim, m.dim_p)},
                                     {inner, heads_map(m.dim, m.dim_p, c0)},
                                     {gn, heads_map(m.state, m.state_p, c0 + m.off_b())},
                                     {gn, heads_map(m.state, m.state_p, c0 + m.off_c())},
                                     {m.heads, at(m.off_dt())}}));
        }
        case CERA_ROLE_SSM_DT_BIAS: return take(S_D, ssm) ? done(vector(L.dt_bias, m.heads)) : misfit();
        case CERA_ROLE_SSM_A_LOG: return take(S_E, ssm) ? done(vector(L.a_log, m.heads)) : misfit();
        case CERA_ROLE_SSM_D: return take(S_F, ssm) ? done(vector(L.skip, m.heads)) : misfit();
        case CERA_ROLE_SSM_NORM: return take(S_G, ssm) ? done(parts(table(L.ssm_norm, 1), {{(size_t)m.heads * m.dim, heads_map(m.dim, m.dim_p)}})) : misfit();
        case CERA_ROLE_FFN_GATE: return take(S_EXPERTS, d.ff == CERA_FF_GATED) ? done(matrix(L.ffn.gate_up, d.ff_width, W, at(0), at(0))) : misfit();
        case CERA_ROLE_FFN_UP: return take(S_EXPERTS + 1, d.ff == CERA_FF_GATED) ? done(matrix(L.ffn.gate_up, d.ff_width, W, at(L.ffn.ff_p), at(0))) : misfit();
        case CERA_ROLE_FFN_DOWN: return take(S_EXPERTS + 2, d.ff == CERA_FF_GATED) ? done(matrix(L.ffn.down, W, d.ff_width, at(0), at(0))) : misfit();
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
        case CERA_ROLE_GRU_Z: return take(S_A, gru) ? done(matrix(L.in, d.recurrent_width, W, at(0), at(0))) : misfit();
        case CERA_ROLE_GRU_X: return take(S_B, gru) ? done(matrix(L.in, d.recurrent_width, W, at(L.wp), at(0))) : misfit();
        case CERA_ROLE_GRU_GATE: return take(S_C, gru) ? done(matrix(L.in, d.recurrent_width, W, at(2 * L.wp), at(0))) : misfit();
        case CERA_ROLE_GRU_Z_BIAS: return take(S_D, gru) ? done(vector(L.z_bias, d.recurrent_width)) : misfit();
        case CERA_ROLE_GRU_X_BIAS: return take(S_E, gru) ? done(vector(L.x_bias, d.recurrent_width)) : misfit();
        case CERA_ROLE_ROUTER: return take(S_ROUTER, d.ff == CERA_FF_MOE) ? done(matrix(L.ffn.router, d.n_experts, W, at(0), at(0))) : misfit();
        default: return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: unknown role %d for layer %d", role, layer);
    }
}

int32_t LayeredModel::add_expert(int32_t role, uint32_t layer, uint32_t expert, int32_t type, size_t rows, size_t cols, const void *bytes, size_t nbytes) {
    if (layer >= cfg.n_layers || layers[layer].d.ff != CERA_FF_MOE || expert >= layers[layer].d.n_experts)
        return fail(CERA_CUDA_ERR_BAD_ARG, "add_expert_tensor: layer %u has no expert %u", layer, expert);
    if (role < CERA_ROLE_EXPERT_GATE || role > CERA_ROLE_EXPERT_DOWN) return fail(CERA_CUDA_ERR_BAD_ARG, "add_expert_tensor: role %d", role);
    LayerWeights &L = layers[layer];
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

// angle = position * base^(-2i / rot), pairs of (cos, sin) per position; worked out in double, kept in f32
int32_t LayeredModel::rope_table(float base, uint32_t rot, const float **out) {
    *out = nullptr;
    if (!rot) return CERA_CUDA_OK;
    for (const Rope &r : ropes)
        if (r.base == base && r.rot == rot) {
            *out = r.table;
            return CERA_CUDA_OK;
        }
    std::vector<float> t((size_t)max_seq_len * rot);
    for (uint32_t i = 0; i < rot / 2; ++i) {
        const double f = std::pow((double)base, -2.0 * i / rot);
        for (size_t p = 0; p < max_seq_len; ++p) {
            t[p * rot + 2 * i] = (float)std::cos((double)p * f);
            t[p * rot + 2 * i + 1] = (float)std::sin((double)p * f);
        }
    }
    Rope r{base, rot, nullptr};
    CERA_TRY(dev_alloc((void **)&r.table, t.size() * 4));
    CERA_CUDA_TRY(cudaMemcpy(r.table, t.data(), t.size() * 4, cudaMemcpyHostToDevice));
    ropes.push_back(r);
    *out = r.table;
    return CERA_CUDA_OK;
}

// Latent attention with expanded keys and values: every head has its own.
AttentionTcShape expanded(const LatentShape &s) { return AttentionTcShape{s.heads, 1, s.dim_p, s.rot_p, s.vdim_p, s.scale, 0.0f}; }

int32_t LayeredModel::build() {
    if (cfg.tied_output) {
        head = embd;
        head_seen = embd_seen;
    }
    if (!embd_seen || !head_seen || !out_norm.g || (cfg.bigram_buckets && !bigram_seen))
        return fail(CERA_CUDA_ERR_STATE, "finalize: an embedding, the head or the final norm is missing");
    for (uint32_t i = 0; i < cfg.n_layers; ++i) {
        const LayerWeights &L = layers[i];
        const bool moe = L.d.ff == CERA_FF_MOE, ff = L.d.ff != CERA_FF_NONE, post = !cfg.no_post_norms;
        const size_t own = S_A + mixer_slots(L.d);
        for (size_t sl = 0; sl < L.seen.size(); ++sl) {
            const bool need = sl == S_PRE || (sl == S_POST && post) || sl == S_OUT || (sl >= S_A && sl < own) || (sl == S_FF_PRE && ff) ||
                              (sl == S_FF_POST && ff && post) || (sl == S_ROUTER && moe) || (sl >= S_EXPERTS && ff);
            if (need && !L.seen[sl]) return fail(CERA_CUDA_ERR_STATE, "finalize: layer %u is missing a tensor (slot %zu)", i, sl);
        }
    }
    const size_t C = LAYERED_CHUNK < max_seq_len ? LAYERED_CHUNK : max_seq_len;
    size_t pre_w = 0, mix_w = 64, q_w = 0, ql = 0, part = 0, heads = 1, gather_w = 0, eo_rows = 0, ff_w = 0, unit_w = 0, experts = 1, used = 1, kx = 0, vx = 0,
           conv_w = 0, aux_w = 0;
    auto up = [](size_t &a, size_t b) { a = a > b ? a : b; };
    ld_v = pad_to(max_seq_len, 64);
    for (auto &L : layers) {
        up(pre_w, L.in.rows);
        up(mix_w, L.out.ld);
        if (L.is(CERA_MIXER_LATENT_ATTENTION)) {
            const LatentShape &s = L.s;
            up(q_w, s.q_ld());
            up(heads, s.heads);
            up(ql, (size_t)s.heads * (s.rank_p + s.rot_p));
            up(part, (size_t)s.heads * (s.rank_p + 2));
            up(kx, (size_t)s.heads * s.dim_p);
            up(vx, (size_t)s.heads * s.vdim_p);
            CERA_TRY(rope_table(L.d.rope_base, s.rot, &L.rope));
        } else if (L.is(CERA_MIXER_ATTENTION)) {
            up(q_w, L.a.q_ld());
            up(part, (size_t)L.a.heads * (L.a.vdim_p + 2));
            CERA_TRY(rope_table(L.d.rope_base, L.a.rot, &L.rope));
        } else if (L.is(CERA_MIXER_RGLRU)) {
            up(conv_w, L.lru.wp);
            up(aux_w, 2 * (size_t)L.lru.wp);
        } else if (L.is(CERA_MIXER_SSM)) {
            up(conv_w, L.ssm.s.channels());
            up(aux_w, L.ssm.s.inner_p());
        }
        if (L.d.ff == CERA_FF_MOE) {
            up(ff_w, L.ffn.ff_p);
            up(experts, L.d.n_experts);
            up(used, L.d.n_used);
            gather_w = ld;
            eo_rows = C * used;
        } else if (L.d.ff == CERA_FF_GATED) {
            up(unit_w, L.ffn.ff_p);
        }
    }
    bool repeats = false;
    for (auto &R : runs) {
        const LayerWeights &L = layers[R.layer];
        repeats |= R.again;
        if (L.is(CERA_MIXER_LATENT_ATTENTION)) {
            CERA_TRY(dev_alloc(&R.cache_a, (size_t)max_seq_len * L.s.rank_p * esz));
            CERA_TRY(dev_alloc(&R.cache_b, (size_t)max_seq_len * L.s.rot_p * esz));
            continue;
        }
        if (L.is(CERA_MIXER_ATTENTION)) {
            const size_t v_bytes = (size_t)L.a.kv_heads * L.a.vdim_p * ld_v * esz;
            CERA_TRY(dev_alloc(&R.cache_a, (size_t)max_seq_len * L.a.kv_heads * L.a.dim_p * esz));
            CERA_TRY(dev_alloc(&R.cache_b, v_bytes));
            // positions never written are multiplied by a zero weight: they must not hold a NaN
            CERA_CUDA_TRY(cudaMemset(R.cache_b, 0, v_bytes));
            continue;
        }
        R.state_n = L.is(CERA_MIXER_RGLRU) ? L.lru.wp : L.is(CERA_MIXER_SSM) ? (size_t)L.ssm.s.inner_p() * L.ssm.s.state_p : L.wp;
        CERA_TRY(vec(&R.state, (uint32_t)R.state_n));
        R.ring_n = L.is(CERA_MIXER_MINGRU) ? 0 : (size_t)L.d.conv_taps * (L.is(CERA_MIXER_RGLRU) ? L.lru.conv : L.ssm.conv).channels;
        if (R.ring_n) CERA_TRY(vec(&R.ring, (uint32_t)R.ring_n));
    }
    CERA_TRY(dev_alloc((void **)&final_hidden, (size_t)ld * 4));
    CERA_TRY(dev_alloc((void **)&x, C * ld * 4));
    if (repeats) CERA_TRY(dev_alloc((void **)&emb, C * ld * 4));
    CERA_TRY(dev_alloc((void **)&y, C * ld * 4));
    CERA_TRY(dev_alloc((void **)&h32, C * ld * 4));
    CERA_TRY(dev_alloc(&h, C * ld * esz));
    CERA_TRY(dev_alloc((void **)&pre, C * pre_w * 4));
    CERA_TRY(dev_alloc(&mix, C * mix_w * esz));  // padding columns meet zero weights: finite is enough
    CERA_CUDA_TRY(cudaMemset(mix, 0, C * mix_w * esz));
    CERA_TRY(dev_alloc((void **)&rows_dev, C * 4));
    if (conv_w) CERA_TRY(dev_alloc(&conv, C * conv_w * esz));
    if (aux_w) CERA_TRY(dev_alloc((void **)&aux, C * aux_w * 4));
    if (has_attention) {
        CERA_TRY(dev_alloc((void **)&q32, C * q_w * 4));
        if (!f32) CERA_TRY(dev_alloc(&qt, C * q_w * esz));
        CERA_TRY(dev_alloc((void **)&lat.part, KV_MAX_SPLITS * part * 4));
    }
    if (ql) {
        CERA_TRY(dev_alloc((void **)&gate, C * heads * 4));
        CERA_TRY(dev_alloc((void **)&lat.q_lat, LATENT_MAX_SPLITS * ql * 4));
        bool fast = false;
        for (auto &L : layers) fast |= !f32 && L.is(CERA_MIXER_LATENT_ATTENTION) && attention_tc_supports(expanded(L.s));
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
        CERA_TRY(dev_alloc((void **)&eo, eo_rows * ld * 4));
    }
    const size_t act_n = eo_rows * ff_w > C * unit_w ? eo_rows * ff_w : C * unit_w;
    if (act_n) CERA_TRY(dev_alloc(&act, act_n * esz));
    rows_alloc = C;
    return CERA_CUDA_OK;
}

RglruView LayeredModel::rglru_view(const LayerRun &R) const {
    RglruView v = layers[R.layer].lru;
    v.state = R.state;
    v.conv.ring = R.ring;
    return v;
}
SsmView LayeredModel::ssm_view(const LayerRun &R) const {
    SsmView v = layers[R.layer].ssm;
    v.state = R.state;
    v.conv.ring = R.ring;
    return v;
}

int32_t LayeredModel::enqueue_step(int kind, uint32_t splits) {
    cudaStream_t st = stream;
    CERA_TRY(launch_embed_dense(embd, bigram, bigram_rule, nullptr, dyn, 1, embedding_scale(), x, emb, st));
    ResidualNorm rn;  // the boundary ahead of the next sublayer
    rn.x = x;
    rn.h = h;
    rn.h_f32 = f32;
    for (auto &R : runs) {
        LayerWeights &L = layers[R.layer];
        rn.pre = L.pre;
        rn.add = R.again ? emb : nullptr;
        CERA_TRY(launch_residual_norm(rn, hidden_size, ld, 1, cfg.norm_eps, st));
        rn.add = nullptr;
        if (L.is(CERA_MIXER_MINGRU)) {
            CERA_TRY(launch_mingru_step(L.in, h, L.z_bias, L.x_bias, R.state, mix, st));
        } else {
            CERA_TRY(launch_dense_gemv(L.in, h, pre, st));
        }
        if (L.is(CERA_MIXER_LATENT_ATTENTION)) {
            CERA_TRY(launch_latent_prepare(pre, L.s, 1, 0, dyn + DYN_POS, L.c_norm, cfg.norm_eps, L.rope, R.cache_a, R.cache_b, f32, q32, nullptr, gate, st));
            CERA_TRY(launch_latent_attention(q32, L.s, L.uk, L.uv, R.cache_a, R.cache_b, L.sink, gate, 1, 0, dyn + DYN_LEN, splits, lat, mix, L.out.ld, st));
        } else if (L.is(CERA_MIXER_ATTENTION)) {
            CERA_TRY(launch_grouped_prepare(pre, L.a, 1, 0, dyn + DYN_POS, L.in_bias, L.rope, R.cache_a, R.cache_b, ld_v, f32, q32, nullptr, st));
            CERA_TRY(launch_grouped_attention(q32, L.a, R.cache_a, R.cache_b, ld_v, f32, 1, 0, dyn + DYN_LEN, splits, lat.part, mix, L.out.ld, st));
        } else if (L.is(CERA_MIXER_RGLRU)) {
            CERA_TRY(launch_rglru_step(pre, rglru_view(R), dyn + DYN_POS, mix, st));
        } else if (L.is(CERA_MIXER_SSM)) {
            const SsmView v = ssm_view(R);
            CERA_TRY(launch_ssm_step(pre, v, dyn + DYN_POS, aux, f32, st));
            CERA_TRY(launch_gated_norm(aux, pre, v, 1, mix, L.out.ld, f32, st));
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
        } else if (L.d.ff == CERA_FF_GATED) {
            rn.pre = L.ff_pre;
            CERA_TRY(launch_residual_norm(rn, hidden_size, ld, 1, cfg.norm_eps, st));
            CERA_TRY(launch_gated_unit_step(L.ffn.gate_up, h, ExpertAct{L.d.act_limit, L.d.act_alpha, L.d.act_shift}, act, st));
            CERA_TRY(launch_dense_gemv(L.ffn.down, act, y, st));
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

// Queries of a portion in groups whose (query, split) pairs fit the scratch: f(first, count, splits).
template <class F>
int32_t in_query_groups(size_t n, size_t start_pos, F f) {
    const uint32_t splits = kv_splits(start_pos + n);
    size_t cn = 0;
    for (size_t j = 0; j < n; j += cn) {
        cn = n - j < KV_MAX_SPLITS ? n - j : KV_MAX_SPLITS;
        uint32_t sp = splits;
        while (sp > 1 && cn * sp > KV_MAX_SPLITS) sp /= 2;
        CERA_TRY(f(j, cn, sp));
    }
    return CERA_CUDA_OK;
}

// The mixer over a chunk: h -> `mix` -> y.
int32_t LayeredModel::mixer_chunk(LayerRun &R, size_t n, size_t start_pos, float *y_out) {
    LayerWeights &L = layers[R.layer];
    DenseGemm g;
    g.w = L.in;
    g.x = h;
    g.n = (uint32_t)n;
    g.out = pre;
    g.ldo = L.in.rows;
    CERA_TRY(launch_dense_gemm(g, stream));
    switch (L.d.mixer) {
        case CERA_MIXER_MINGRU: CERA_TRY(launch_mingru_scan(pre, n, L.wp, L.z_bias, L.x_bias, R.state, mix, f32, stream)); break;
        case CERA_MIXER_LATENT_ATTENTION: CERA_TRY(latent_chunk(R, n, start_pos)); break;
        case CERA_MIXER_ATTENTION: CERA_TRY(attention_chunk(R, n, start_pos)); break;
        case CERA_MIXER_RGLRU: CERA_TRY(rglru_chunk(R, n, start_pos)); break;
        default: CERA_TRY(ssm_chunk(R, n, start_pos)); break;
    }
    DenseGemm o;
    o.w = L.out;
    o.x = mix;
    o.n = (uint32_t)n;
    o.out = y_out;
    o.ldo = ld;
    return launch_dense_gemm(o, stream);
}

int32_t LayeredModel::attention_chunk(LayerRun &R, size_t n, size_t start_pos) {
    const LayerWeights &L = layers[R.layer];
    const GroupedShape &a = L.a;
    const size_t ldm = L.out.ld;
    const AttentionTcShape tc{a.heads, a.heads / a.kv_heads, a.dim_p, 0, a.vdim_p, a.scale, a.softcap};
    const bool tiles = !f32 && n >= ATTENTION_TC_MIN && attention_tc_supports(tc);
    CERA_TRY(launch_grouped_prepare(pre, a, n, start_pos, nullptr, L.in_bias, L.rope, R.cache_a, R.cache_b, ld_v, f32, tiles ? nullptr : q32, tiles ? qt : nullptr,
                                    stream));
    if (tiles) {
        AttentionTcOperands o;
        o.q = qt;
        o.k = R.cache_a;
        o.v = R.cache_b;
        o.positions = max_seq_len;
        o.ld_v = ld_v;
        return launch_attention_tc(tc, o, n, start_pos, mix, ldm, stream);
    }
    return in_query_groups(n, start_pos, [&](size_t j, size_t cn, uint32_t sp) {
        return launch_grouped_attention(q32 + j * a.q_ld(), a, R.cache_a, R.cache_b, ld_v, f32, cn, start_pos + j, nullptr, sp, lat.part,
                                        (char *)mix + j * ldm * esz, ldm, stream);
    });
}

int32_t LayeredModel::rglru_chunk(LayerRun &R, size_t n, size_t start_pos) {
    const RglruView v = rglru_view(R);
    CERA_TRY(launch_conv(pre + v.wp, 2 * (size_t)v.wp, v.in_bias + v.wp, v.conv, 0, n, start_pos, conv, v.wp, f32, stream));
    DenseGemm g;
    g.w = v.gates;
    g.x = conv;
    g.n = (uint32_t)n;
    g.out = aux;
    g.ldo = 2 * (size_t)v.wp;
    g.block_rows = 2 * v.block_p;
    g.x_ld = v.wp;
    CERA_TRY(launch_dense_gemm(g, stream));
    return launch_rglru_scan(pre, conv, aux, v, n, start_pos, mix, f32, stream);
}

int32_t LayeredModel::ssm_chunk(LayerRun &R, size_t n, size_t start_pos) {
    const SsmView v = ssm_view(R);
    const uint32_t channels = v.s.channels();
    CERA_TRY(launch_conv(pre + v.s.inner_p(), v.s.in_p, nullptr, v.conv, 1, n, start_pos, conv, channels, f32, stream));
    if (!f32 && n >= SSM_CHUNK_MIN && ssm_chunks_support(v.s)) CERA_TRY(launch_ssm_chunks(pre, conv, v, n, start_pos, aux, stream));
    else CERA_TRY(launch_ssm_scan(pre, conv, v, n, start_pos, aux, f32, stream));
    return launch_gated_norm(aux, pre, v, n, mix, layers[R.layer].out.ld, f32, stream);
}

int32_t LayeredModel::latent_chunk(LayerRun &R, size_t n, size_t start_pos) {
    const LayerWeights &L = layers[R.layer];
    const LatentShape &s = L.s;
    const size_t ldm = L.out.ld;
    const bool expand = !f32 && n >= ATTENTION_TC_MIN && k_exp && attention_tc_supports(expanded(s));
    CERA_TRY(launch_latent_prepare(pre, s, n, start_pos, nullptr, L.c_norm, cfg.norm_eps, L.rope, R.cache_a, R.cache_b, f32, expand ? nullptr : q32,
                                   expand ? qt : nullptr, gate, stream));
    if (expand) {
        DenseGemm k;
        k.w = L.uk;
        k.x = R.cache_a;
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
        AttentionTcOperands t;
        t.q = qt;
        t.k = k_exp;
        t.k_rot = R.cache_b;
        t.v = v_exp;
        t.positions = max_seq_len;
        t.ld_v = exp_rows;
        t.sink = L.sink;
        t.gate = gate;
        return launch_attention_tc(expanded(s), t, n, start_pos, mix, ldm, stream);
    }
    return in_query_groups(n, start_pos, [&](size_t j, size_t cn, uint32_t sp) {
        return launch_latent_attention(q32 + j * s.q_ld(), s, L.uk, L.uv, R.cache_a, R.cache_b, L.sink, gate + j * s.heads, cn, start_pos + j, nullptr, sp, lat,
                                       (char *)mix + j * ldm * esz, ldm, stream);
    });
}

// The routed feed-forward over a chunk: h, h32 -> `eo` in bucket order; `next` sums the picks.
int32_t LayeredModel::experts_chunk(LayerWeights &L, size_t n, ResidualNorm *next) {
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

// The gated unit over a chunk: h -> y.
int32_t LayeredModel::unit_chunk(LayerWeights &L, size_t n, ResidualNorm *next) {
    DenseGemm g;
    g.w = L.ffn.gate_up;
    g.x = h;
    g.n = (uint32_t)n;
    g.out_kind = DENSE_GATED_UNIT;
    g.out = act;
    g.ldo = L.ffn.ff_p;
    g.act = ExpertAct{L.d.act_limit, L.d.act_alpha, L.d.act_shift};
    CERA_TRY(launch_dense_gemm(g, stream));
    DenseGemm o;
    o.w = L.ffn.down;
    o.x = act;
    o.n = (uint32_t)n;
    o.out = y;
    o.ldo = ld;
    CERA_TRY(launch_dense_gemm(o, stream));
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
    CERA_TRY(launch_embed_dense(embd, bigram, bigram_rule, pf_tokens, nullptr, n, embedding_scale(), x, emb, st));
    ResidualNorm rn;
    rn.x = x;
    rn.h = h;
    rn.h_f32 = f32;
    for (auto &R : runs) {
        LayerWeights &L = layers[R.layer];
        rn.pre = L.pre;
        rn.add = R.again ? emb : nullptr;
        CERA_TRY(launch_residual_norm(rn, hidden_size, ld, n, cfg.norm_eps, st));
        rn.add = nullptr;
        CERA_TRY(mixer_chunk(R, n, start_pos, y));
        rn.y = y;
        rn.entry_of = nullptr;
        rn.post = L.post;
        if (L.d.ff == CERA_FF_MOE) {
            rn.pre = L.ff_pre;
            rn.h32 = h32;
            CERA_TRY(launch_residual_norm(rn, hidden_size, ld, n, cfg.norm_eps, st));
            rn.h32 = nullptr;
            CERA_TRY(experts_chunk(L, n, &rn));
        } else if (L.d.ff == CERA_FF_GATED) {
            rn.pre = L.ff_pre;
            CERA_TRY(launch_residual_norm(rn, hidden_size, ld, n, cfg.norm_eps, st));
            CERA_TRY(unit_chunk(L, n, &rn));
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
    // cached positions beyond len are overwritten later; a recurrent state exists for the current position only
    if (len && has_recurrence)
        return fail(CERA_CUDA_ERR_UNSUPPORTED, "truncate_kv: recurrent layers keep no state of position %zu (restore a snapshot, or truncate to 0)", len);
    if (!finalized) return CERA_CUDA_OK;
    if (len == 0)
        for (auto &R : runs) {
            if (R.state) CERA_CUDA_TRY(cudaMemsetAsync(R.state, 0, R.state_n * 4, stream));
            if (R.ring) CERA_CUDA_TRY(cudaMemsetAsync(R.ring, 0, R.ring_n * 4, stream));
        }
    return check_cuda(cudaStreamSynchronize(stream), "truncate_kv");
}

struct LayeredSnapshot {
    uint32_t magic, version, n_layers, elem_bytes;
    uint64_t seq_len, bytes;
};
constexpr uint32_t LAYERED_MAGIC = 0x4C4B4243u;  // "CBKL"

std::vector<LayeredModel::Piece> LayeredModel::pieces(size_t n) const {
    std::vector<Piece> out;
    for (const auto &R : runs) {
        const LayerWeights &L = layers[R.layer];
        if (L.is(CERA_MIXER_LATENT_ATTENTION)) {
            out.push_back({R.cache_a, n * L.s.rank_p * esz, 1, 0});
            out.push_back({R.cache_b, n * L.s.rot_p * esz, 1, 0});
        } else if (L.is(CERA_MIXER_ATTENTION)) {
            out.push_back({R.cache_a, n * L.a.kv_heads * L.a.dim_p * esz, 1, 0});
            out.push_back({R.cache_b, n * esz, (size_t)L.a.kv_heads * L.a.vdim_p, ld_v * esz});
        } else {
            out.push_back({R.state, R.state_n * 4, 1, 0});
            if (R.ring) out.push_back({R.ring, R.ring_n * 4, 1, 0});
        }
    }
    return out;
}

// header, the consumed tokens, then per layer run its cached positions or its state
size_t LayeredModel::snapshot_bytes() const {
    size_t n = sizeof(LayeredSnapshot) + seq_len * 4;
    for (const Piece &q : pieces(seq_len)) n += q.bytes * q.rows;
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
    for (const Piece &q : pieces(seq_len)) {
        if (!q.bytes) continue;
        CERA_CUDA_TRY(cudaMemcpy2D(p, q.bytes, q.p, q.rows > 1 ? q.pitch : q.bytes, q.bytes, q.rows, cudaMemcpyDeviceToHost));
        p += q.bytes * q.rows;
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
    for (const Piece &q : pieces(n)) need += q.bytes * q.rows;
    if (bytes != need || hd.bytes != need) return fail(CERA_CUDA_ERR_BAD_ARG, "kv_restore: %zu bytes, %zu expected", bytes, need);
    CERA_CUDA_TRY(cudaStreamSynchronize(stream));
    const char *p = (const char *)data + sizeof(hd);
    history.assign((const uint32_t *)p, (const uint32_t *)p + n);
    p += n * 4;
    for (const Piece &q : pieces(n)) {
        if (!q.bytes) continue;
        CERA_CUDA_TRY(cudaMemcpy2D(q.p, q.rows > 1 ? q.pitch : q.bytes, p, q.bytes, q.bytes, q.rows, cudaMemcpyHostToDevice));
        p += q.bytes * q.rows;
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
    } else if (d.mixer == CERA_MIXER_ATTENTION) {
        if (!d.n_heads || !d.n_kv_heads || d.n_heads % d.n_kv_heads || !d.head_dim || !d.value_dim || d.rot_dim % 2 || d.rot_dim > d.head_dim ||
            (d.rot_dim && !(d.rope_base > 0.0f)) || d.softcap < 0.0f)
            return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: layer %u: attention sizes", i);
        if (d.head_dim > 1024 || d.value_dim > 1024) return fail(CERA_CUDA_ERR_UNSUPPORTED, "model_create: layer %u: heads of %u / %u (at most 1024)", i, d.head_dim, d.value_dim);
    } else if (d.mixer == CERA_MIXER_RGLRU) {
        if (!d.recurrent_width || !d.n_blocks || d.recurrent_width % d.n_blocks || !d.conv_taps)
            return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: layer %u: %u channels in %u blocks, %u taps", i, d.recurrent_width, d.n_blocks, d.conv_taps);
        if (d.recurrent_width / d.n_blocks > 8192) return fail(CERA_CUDA_ERR_UNSUPPORTED, "model_create: layer %u: blocks of more than 8192 channels", i);
    } else if (d.mixer == CERA_MIXER_SSM) {
        if (!d.n_heads || !d.value_dim || !d.state_size || !d.n_groups || d.n_heads % d.n_groups || !d.n_norm_groups || !d.conv_taps ||
            (uint64_t)d.n_heads * d.value_dim % d.n_norm_groups)
            return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: layer %u: state-space sizes", i);
        if (d.state_size > SSM_MAX_STATE) return fail(CERA_CUDA_ERR_UNSUPPORTED, "model_create: layer %u: state of %u (at most %u)", i, d.state_size, SSM_MAX_STATE);
    } else {
        return fail(CERA_CUDA_ERR_UNSUPPORTED, "model_create: layer %u: unknown mixer %d", i, d.mixer);
    }
    if (d.ff == CERA_FF_NONE) return CERA_CUDA_OK;
    if (d.ff == CERA_FF_GATED) return d.ff_width ? CERA_CUDA_OK : fail(CERA_CUDA_ERR_BAD_ARG, "model_create: layer %u: feed-forward width is zero", i);
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
    if (c.loop_times > 1 && (c.loop_start >= c.loop_stop || c.loop_stop > c.n_layers))
        return fail(CERA_CUDA_ERR_BAD_ARG, "model_create: layers %u to %u repeat, of %u", c.loop_start, c.loop_stop, c.n_layers);
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
