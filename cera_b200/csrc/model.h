// The model object behind cera_cuda_model: what every architecture shares, and what one has to provide.
//
// The base owns the sequence (position counter, the tokens consumed so far), the decode step's CUDA graphs and the
// device words they read (token, position, previous token), the logits and token buffers, and the loops over prompt
// chunks and generated tokens.  An architecture (llama.cu, layered.cu) derives from it and supplies its weights, its
// per-sequence state and two enqueue functions: one decode step, one chunk of a prompt.
#pragma once

#include <map>
#include <mutex>
#include <vector>

#include "common.cuh"

namespace cera {

// What a recorded decode step ends with: nothing (the token only extends the state), logits, a greedy pick, or a
// greedy pick that feeds the next step.
enum GraphKind { G_BODY = 0, G_LOGITS = 1, G_GREEDY = 2, G_CHAIN = 3 };

// Words of cera_cuda_model::dyn.
enum { DYN_TOKEN = 0, DYN_POS = 1, DYN_LEN = 2, DYN_STEP = 3, DYN_PREV = 4, DYN_WORDS = 5 };
constexpr uint32_t NO_TOKEN = 0xFFFFFFFFu;  // DYN_PREV of a sequence's first token

struct DeviceGuard {
    int prev = 0;
    explicit DeviceGuard(int dev) {
        cudaGetDevice(&prev);
        cudaSetDevice(dev);
    }
    ~DeviceGuard() { cudaSetDevice(prev); }
};

}  // namespace cera

struct cera_cuda_model {
    cera_cuda_model(uint32_t vocab, uint32_t hidden, uint32_t max_seq, int dev)
        : vocab_size(vocab), hidden_size(hidden), max_seq_len(max_seq), device(dev) {}
    virtual ~cera_cuda_model();
    cera_cuda_model(const cera_cuda_model &) = delete;
    cera_cuda_model &operator=(const cera_cuda_model &) = delete;

    const uint32_t vocab_size, hidden_size, max_seq_len;
    const int device;
    std::mutex mu;
    bool finalized = false;
    std::vector<void *> owned;  // plain device allocations to free
    size_t mem_bytes = 0;
    float *logits = nullptr;        // device: logits of the last token
    float *final_hidden = nullptr;  // device: normed hidden state of the last token
    float *pf_logits = nullptr;     // device: logits of several positions, allocated by the first call that asks for them
    uint32_t *argmax_scratch = nullptr;
    uint32_t *dyn = nullptr;       // device: the words the recorded step reads
    uint32_t *tok_out = nullptr;   // device
    uint32_t *h_dyn = nullptr;     // pinned host mirror of dyn, then the returned token
    float *h_logits = nullptr;     // pinned host staging for logits
    uint32_t *pf_tokens = nullptr;  // device: a prompt chunk's token ids
    uint32_t *tok_hist = nullptr;  // device ring of generated tokens (chained greedy decode)
    uint32_t tok_hist_cap = 0;
    cudaStream_t stream = nullptr;
    std::map<uint32_t, cudaGraphExec_t> graphs;  // key = kind | plan << 8
    size_t seq_len = 0;
    std::vector<uint32_t> history;  // the tokens at positions [0, seq_len), NO_TOKEN where unknown
    uint64_t launches = 0;         // kernels launched by decode steps
    uint32_t nodes_per_step[4] = {0, 0, 0, 0};

    // ---- what an architecture provides ------------------------------------------------------------------------
    virtual int32_t add_tensor(int32_t role, int32_t layer, int32_t type, size_t rows, size_t cols, const void *bytes, size_t nbytes) = 0;
    virtual int32_t build() = 0;  // finalize: every tensor is there; allocate state and scratch
    virtual size_t chunk_tokens() const = 0;
    virtual uint32_t plan(size_t n_positions) const = 0;  // launch plan of a decode step over n_positions, part of the graph key
    virtual int32_t enqueue_step(int kind, uint32_t plan) = 0;
    virtual bool batched(size_t n) const = 0;  // does a prompt portion of n tokens take the batched kernels?
    // one chunk (n <= chunk_tokens()) of prompt tokens, all layers; the hidden states of the chunk stay on the device
    virtual int32_t prefill_chunk(const uint32_t *tokens, size_t n, size_t start_pos) = 0;
    virtual int32_t logits_of_last(size_t n) = 0;  // final norm + head of the chunk's last row, into `logits`
    // logits of chunk rows rows[0..n_rows) (null: of all n rows) to host memory, asynchronous on `stream`
    virtual int32_t logits_of_rows(const uint32_t *rows, size_t n_rows, size_t n, float *out) = 0;
    virtual int32_t ready(const char *) { return CERA_CUDA_OK; }  // may a forward call start?
    virtual int32_t after_sync() { return CERA_CUDA_OK; }         // looked at after a synchronisation
    virtual int32_t run_prompt(const uint32_t *tokens, size_t n, size_t start_pos, bool want_logits);
    virtual int32_t rewind(size_t len) = 0;  // drop state beyond position len < seq_len
    virtual size_t snapshot_bytes() const = 0;
    virtual int32_t snapshot(void *out, size_t out_bytes) = 0;
    virtual int32_t restore(const void *data, size_t bytes) = 0;  // sets seq_len and history

    // ---- shared machinery (model.cu) ---------------------------------------------------------------------------
    int32_t dev_alloc(void **p, size_t bytes);
    int32_t alloc_common();  // the buffers above that the architecture has not placed itself
    int32_t get_graph(int kind, uint32_t plan, cudaGraphExec_t *out);
    int32_t run_token(uint32_t token, size_t pos, int kind);
    int32_t launch_advance();  // the chained step's last kernel: this pick becomes the next step's token
    void drop_graphs();
    uint32_t token_before(size_t pos) const { return pos == 0 || pos > history.size() ? cera::NO_TOKEN : history[pos - 1]; }
    int32_t check_portion(const char *what, const uint32_t *tokens, size_t n, size_t start_pos);
};
