// Entry points of the model object that do not depend on the architecture, and the machinery they share: the decode
// step as a CUDA graph per (kind, plan), prompt chunks, the device-chained greedy loop, sequence bookkeeping.
// (cera/src/model/mod.rs:200-606 `trait Model`; cera/src/session.rs:1788-2310 the greedy loop.)
#include "model.h"

#include <cstring>

#include "ops.h"

using namespace cera;

namespace {

// After the argmax of a chained step: record the token, make it the next input, advance the position.
__global__ void advance_kernel(uint32_t *dyn, const uint32_t *tok_out, uint32_t *hist, uint32_t cap) {
    pdl_trigger();
    pdl_wait();
    const uint32_t t = *tok_out, step = dyn[DYN_STEP];
    if (step < cap) hist[step] = t;
    dyn[DYN_PREV] = dyn[DYN_TOKEN];
    dyn[DYN_TOKEN] = t;
    dyn[DYN_POS] += 1;
    dyn[DYN_LEN] += 1;
    dyn[DYN_STEP] = step + 1;
}

}  // namespace

cera_cuda_model::~cera_cuda_model() {
    DeviceGuard dg(device);
    if (stream) cudaStreamSynchronize(stream);
    drop_graphs();
    for (void *p : owned) cudaFree(p);
    if (h_dyn) cudaFreeHost(h_dyn);
    if (h_logits) cudaFreeHost(h_logits);
    if (stream) cudaStreamDestroy(stream);
}

void cera_cuda_model::drop_graphs() {
    for (auto &kv : graphs) cudaGraphExecDestroy(kv.second);
    graphs.clear();
}

int32_t cera_cuda_model::dev_alloc(void **p, size_t bytes) {
    CERA_CUDA_TRY(cudaMalloc(p, bytes));
    owned.push_back(*p);
    mem_bytes += bytes;
    return CERA_CUDA_OK;
}

int32_t cera_cuda_model::alloc_common() {
    if (!logits) CERA_TRY(dev_alloc((void **)&logits, (size_t)vocab_size * 4));
    if (!final_hidden) CERA_TRY(dev_alloc((void **)&final_hidden, (size_t)hidden_size * 4));
    CERA_TRY(dev_alloc((void **)&pf_tokens, (chunk_tokens() + 1) * 4));
    CERA_TRY(dev_alloc((void **)&argmax_scratch, argmax_scratch_words() * 4));
    CERA_TRY(dev_alloc((void **)&dyn, 8 * 4));
    CERA_TRY(dev_alloc((void **)&tok_out, 4));
    tok_hist_cap = max_seq_len;
    CERA_TRY(dev_alloc((void **)&tok_hist, (size_t)tok_hist_cap * 4));
    CERA_CUDA_TRY(cudaMallocHost((void **)&h_dyn, 8 * 4));
    CERA_CUDA_TRY(cudaMallocHost((void **)&h_logits, (size_t)vocab_size * 4));
    CERA_CUDA_TRY(cudaStreamCreateWithFlags(&stream, cudaStreamNonBlocking));
    return check_cuda(cudaDeviceSynchronize(), "finalize");
}

int32_t cera_cuda_model::launch_advance() {
    count_launch();
    return check_cuda(launch_k(advance_kernel, dim3(1), dim3(1), 0, stream, dyn, (const uint32_t *)tok_out, tok_hist, tok_hist_cap), "advance launch");
}

int32_t cera_cuda_model::get_graph(int kind, uint32_t plan, cudaGraphExec_t *out) {
    const uint32_t key = (uint32_t)kind | (plan << 8);
    auto it = graphs.find(key);
    if (it != graphs.end()) {
        *out = it->second;
        return CERA_CUDA_OK;
    }
    const uint64_t before = launches_so_far();
    CERA_CUDA_TRY(cudaStreamBeginCapture(stream, cudaStreamCaptureModeThreadLocal));
    int32_t st = enqueue_step(kind, plan);
    cudaGraph_t graph = nullptr;
    cudaError_t e = cudaStreamEndCapture(stream, &graph);
    if (st != CERA_CUDA_OK) {
        if (graph) cudaGraphDestroy(graph);
        return st;
    }
    CERA_CUDA_TRY(e);
    nodes_per_step[kind] = (uint32_t)(launches_so_far() - before);
    cudaGraphExec_t exec = nullptr;
    e = cudaGraphInstantiate(&exec, graph, 0);
    cudaGraphDestroy(graph);
    CERA_CUDA_TRY(e);
    graphs[key] = exec;
    *out = exec;
    return CERA_CUDA_OK;
}

// Runs one token; leaves results in device buffers (logits / tok_out).
int32_t cera_cuda_model::run_token(uint32_t token, size_t pos, int kind) {
    if (!finalized) return fail(CERA_CUDA_ERR_STATE, "forward: model_finalize has not been called");
    if (token >= vocab_size) return fail(CERA_CUDA_ERR_BAD_ARG, "forward: token %u out of range (vocab %u)", token, vocab_size);
    if (pos != seq_len) return fail(CERA_CUDA_ERR_STATE, "forward: pos %zu != seq_len %zu", pos, seq_len);
    if (pos >= max_seq_len) return fail(CERA_CUDA_ERR_BAD_ARG, "forward: pos %zu exceeds max_seq_len %u", pos, max_seq_len);
    CERA_TRY(ready("forward"));
    cudaGraphExec_t g = nullptr;
    CERA_TRY(get_graph(kind, plan(pos + 1), &g));
    h_dyn[DYN_TOKEN] = token;
    h_dyn[DYN_POS] = (uint32_t)pos;
    h_dyn[DYN_LEN] = (uint32_t)pos + 1;
    h_dyn[DYN_STEP] = 0;
    h_dyn[DYN_PREV] = token_before(pos);
    CERA_CUDA_TRY(cudaMemcpyAsync(dyn, h_dyn, DYN_WORDS * sizeof(uint32_t), cudaMemcpyHostToDevice, stream));
    CERA_CUDA_TRY(cudaGraphLaunch(g, stream));
    launches += nodes_per_step[kind];
    seq_len = pos + 1;
    history.push_back(token);
    return CERA_CUDA_OK;
}

int32_t cera_cuda_model::run_prompt(const uint32_t *tokens, size_t n, size_t start_pos, bool want_logits) {
    if (!batched(n)) {
        // Decode arithmetic for every prompt position (one graph launch per token).  h_dyn is rewritten per
        // token, so wait for the copy of the previous one before touching it again.
        for (size_t i = 0; i < n; ++i) {
            const bool last = i + 1 == n;
            CERA_TRY(run_token(tokens[i], start_pos + i, last && want_logits ? G_LOGITS : G_BODY));
            CERA_CUDA_TRY(cudaStreamSynchronize(stream));
        }
        return after_sync();
    }
    // Batched kernels, one chunk at a time (the reference's ubatch loop, cera/src/model/mod.rs:303-332).
    size_t cn = 0;
    for (size_t done = 0; done < n; done += cn) {
        cn = n - done < chunk_tokens() ? n - done : chunk_tokens();
        CERA_TRY(prefill_chunk(tokens + done, cn, start_pos + done));
        CERA_CUDA_TRY(cudaStreamSynchronize(stream));  // the host token slice may go away after the call
        seq_len = start_pos + done + cn;
        history.insert(history.end(), tokens + done, tokens + done + cn);
    }
    return want_logits ? logits_of_last(cn) : CERA_CUDA_OK;
}

int32_t cera_cuda_model::check_portion(const char *what, const uint32_t *tokens, size_t n, size_t start_pos) {
    if (!finalized) return fail(CERA_CUDA_ERR_STATE, "%s: model_finalize has not been called", what);
    if (start_pos != seq_len) return fail(CERA_CUDA_ERR_STATE, "%s: start_pos %zu != seq_len %zu", what, start_pos, seq_len);
    if (start_pos + n > max_seq_len)
        return fail(CERA_CUDA_ERR_BAD_ARG, "%s: %zu tokens from %zu exceed max_seq_len %u", what, n, start_pos, max_seq_len);
    for (size_t i = 0; i < n; ++i)
        if (tokens[i] >= vocab_size) return fail(CERA_CUDA_ERR_BAD_ARG, "%s: token %u out of range (vocab %u)", what, tokens[i], vocab_size);
    return ready(what);
}

extern "C" {

int32_t cera_cuda_model_add_tensor(cera_cuda_model *m, int32_t role, int32_t layer, int32_t type, size_t rows,
                                   size_t cols, const void *bytes, size_t nbytes) {
    if (!m || !bytes) return fail(CERA_CUDA_ERR_BAD_ARG, "add_tensor: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    if (m->finalized) return fail(CERA_CUDA_ERR_STATE, "add_tensor: model already finalized");
    return m->add_tensor(role, layer, type, rows, cols, bytes, nbytes);
}

int32_t cera_cuda_model_finalize(cera_cuda_model *m) {
    if (!m) return fail(CERA_CUDA_ERR_BAD_ARG, "finalize: null model");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    if (m->finalized) return CERA_CUDA_OK;
    CERA_TRY(m->build());
    CERA_TRY(m->alloc_common());
    m->finalized = true;
    return CERA_CUDA_OK;
}

int32_t cera_cuda_forward(cera_cuda_model *m, uint32_t token, size_t pos, float *logits_out) {
    if (!m || !logits_out) return fail(CERA_CUDA_ERR_BAD_ARG, "forward: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    CERA_TRY(m->run_token(token, pos, G_LOGITS));
    const size_t bytes = (size_t)m->vocab_size * 4;
    CERA_CUDA_TRY(cudaMemcpyAsync(m->h_logits, m->logits, bytes, cudaMemcpyDeviceToHost, m->stream));
    CERA_CUDA_TRY(cudaStreamSynchronize(m->stream));
    CERA_TRY(m->after_sync());
    memcpy(logits_out, m->h_logits, bytes);
    return CERA_CUDA_OK;
}

int32_t cera_cuda_forward_greedy(cera_cuda_model *m, uint32_t token, size_t pos, uint32_t *token_out) {
    if (!m || !token_out) return fail(CERA_CUDA_ERR_BAD_ARG, "forward_greedy: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    CERA_TRY(m->run_token(token, pos, G_GREEDY));
    CERA_CUDA_TRY(cudaMemcpyAsync(m->h_dyn + DYN_WORDS, m->tok_out, 4, cudaMemcpyDeviceToHost, m->stream));
    CERA_CUDA_TRY(cudaStreamSynchronize(m->stream));
    CERA_TRY(m->after_sync());
    *token_out = m->h_dyn[DYN_WORDS];
    return CERA_CUDA_OK;
}

int32_t cera_cuda_forward_prefill(cera_cuda_model *m, const uint32_t *tokens, size_t n, size_t start_pos,
                                  float *logits_out) {
    if (!m || (!tokens && n)) return fail(CERA_CUDA_ERR_BAD_ARG, "forward_prefill: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    if (start_pos != m->seq_len) return fail(CERA_CUDA_ERR_STATE, "forward_prefill: start_pos %zu != seq_len %zu", start_pos, m->seq_len);
    if (n == 0) return CERA_CUDA_OK;
    CERA_TRY(m->check_portion("forward_prefill", tokens, n, start_pos));
    CERA_TRY(m->run_prompt(tokens, n, start_pos, logits_out != nullptr));
    if (logits_out) {
        const size_t bytes = (size_t)m->vocab_size * 4;
        CERA_CUDA_TRY(cudaMemcpyAsync(m->h_logits, m->logits, bytes, cudaMemcpyDeviceToHost, m->stream));
        CERA_CUDA_TRY(cudaStreamSynchronize(m->stream));
        memcpy(logits_out, m->h_logits, bytes);
    }
    return CERA_CUDA_OK;
}

// A prompt portion with the logits of chosen positions: rows want[0..n_want) in ascending order (null: every position),
// out[.][vocab] on the host, token-major.  Model::forward_prefill_logits_all (cera/src/model/mod.rs:507-533, used by
// speculative decoding) is the case of every position.
int32_t cera_cuda_forward_prefill_logits_at(cera_cuda_model *m, const uint32_t *tokens, size_t n, size_t start_pos, const uint32_t *want,
                                            size_t n_want, float *logits_out) {
    if (!m || !tokens || (!logits_out && (!want || n_want))) return fail(CERA_CUDA_ERR_BAD_ARG, "forward_prefill_logits_at: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    CERA_TRY(m->check_portion("forward_prefill_logits_at", tokens, n, start_pos));
    const size_t vocab = m->vocab_size;
    if (!want) n_want = n;
    for (size_t i = 0; want && i < n_want; ++i)
        if (want[i] >= n || (i && want[i] <= want[i - 1]))
            return fail(CERA_CUDA_ERR_BAD_ARG, "forward_prefill_logits_at: position %u of %zu tokens is outside or out of order", want[i], n);
    size_t at = 0;  // wanted positions served so far
    if (!m->batched(n)) {
        for (size_t i = 0; i < n; ++i) {
            const bool wanted = at < n_want && (want ? want[at] : at) == i;
            CERA_TRY(m->run_token(tokens[i], start_pos + i, wanted ? G_LOGITS : G_BODY));
            if (wanted) CERA_CUDA_TRY(cudaMemcpyAsync(logits_out + at++ * vocab, m->logits, vocab * 4, cudaMemcpyDeviceToHost, m->stream));
            CERA_CUDA_TRY(cudaStreamSynchronize(m->stream));
        }
        return m->after_sync();
    }
    std::vector<uint32_t> rows;
    size_t cn = 0;
    for (size_t done = 0; done < n; done += cn) {
        cn = n - done < m->chunk_tokens() ? n - done : m->chunk_tokens();
        CERA_TRY(m->prefill_chunk(tokens + done, cn, start_pos + done));
        rows.clear();
        for (; want && at + rows.size() < n_want && want[at + rows.size()] < done + cn;) rows.push_back(want[at + rows.size()] - (uint32_t)done);
        const size_t got = want ? rows.size() : cn;
        if (got) CERA_TRY(m->logits_of_rows(want ? rows.data() : nullptr, got, cn, logits_out + at * vocab));
        at += got;
        CERA_CUDA_TRY(cudaStreamSynchronize(m->stream));
        m->seq_len = start_pos + done + cn;
        m->history.insert(m->history.end(), tokens + done, tokens + done + cn);
    }
    return CERA_CUDA_OK;
}

int32_t cera_cuda_forward_prefill_logits_all(cera_cuda_model *m, const uint32_t *tokens, size_t n, size_t start_pos,
                                             float *logits_out) {
    if (!logits_out) return fail(CERA_CUDA_ERR_BAD_ARG, "forward_prefill_logits_all: null argument");
    return cera_cuda_forward_prefill_logits_at(m, tokens, n, start_pos, nullptr, 0, logits_out);
}

int32_t cera_cuda_generate_greedy(cera_cuda_model *m, uint32_t first_token, size_t start_pos, size_t n,
                                  uint32_t *tokens_out, float *device_ms) {
    if (!m || !tokens_out) return fail(CERA_CUDA_ERR_BAD_ARG, "generate_greedy: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    if (!m->finalized) return fail(CERA_CUDA_ERR_STATE, "generate_greedy: model_finalize has not been called");
    if (first_token >= m->vocab_size) return fail(CERA_CUDA_ERR_BAD_ARG, "generate_greedy: token out of range");
    if (start_pos != m->seq_len) return fail(CERA_CUDA_ERR_STATE, "generate_greedy: start_pos %zu != seq_len %zu", start_pos, m->seq_len);
    if (start_pos + n > m->max_seq_len) return fail(CERA_CUDA_ERR_BAD_ARG, "generate_greedy: %zu tokens from %zu exceed max_seq_len %u", n, start_pos, m->max_seq_len);
    CERA_TRY(m->ready("generate_greedy"));
    if (n == 0) return CERA_CUDA_OK;
    m->h_dyn[DYN_TOKEN] = first_token;
    m->h_dyn[DYN_POS] = (uint32_t)start_pos;
    m->h_dyn[DYN_LEN] = (uint32_t)start_pos + 1;
    m->h_dyn[DYN_STEP] = 0;
    m->h_dyn[DYN_PREV] = m->token_before(start_pos);
    CERA_CUDA_TRY(cudaMemcpyAsync(m->dyn, m->h_dyn, DYN_WORDS * sizeof(uint32_t), cudaMemcpyHostToDevice, m->stream));
    cudaEvent_t e0 = nullptr, e1 = nullptr;
    CERA_CUDA_TRY(cudaEventCreate(&e0));
    CERA_CUDA_TRY(cudaEventCreate(&e1));
    // instantiate every graph the run needs before the timed region
    for (size_t i = 0; i < n; ++i) {
        cudaGraphExec_t g = nullptr;
        CERA_TRY(m->get_graph(G_CHAIN, m->plan(start_pos + i + 1), &g));
    }
    CERA_CUDA_TRY(cudaEventRecord(e0, m->stream));
    for (size_t i = 0; i < n; ++i) {
        cudaGraphExec_t g = nullptr;
        CERA_TRY(m->get_graph(G_CHAIN, m->plan(start_pos + i + 1), &g));
        CERA_CUDA_TRY(cudaGraphLaunch(g, m->stream));
    }
    CERA_CUDA_TRY(cudaEventRecord(e1, m->stream));
    m->launches += (uint64_t)m->nodes_per_step[G_CHAIN] * n;
    m->seq_len = start_pos + n;
    CERA_CUDA_TRY(cudaMemcpyAsync(tokens_out, m->tok_hist, n * 4, cudaMemcpyDeviceToHost, m->stream));
    CERA_CUDA_TRY(cudaStreamSynchronize(m->stream));
    float ms = 0.0f;
    CERA_CUDA_TRY(cudaEventElapsedTime(&ms, e0, e1));
    if (device_ms) *device_ms = ms;
    cudaEventDestroy(e0);
    cudaEventDestroy(e1);
    m->history.push_back(first_token);
    m->history.insert(m->history.end(), tokens_out, tokens_out + n - 1);  // the last pick has not been consumed
    return m->after_sync();
}

int32_t cera_cuda_truncate_kv(cera_cuda_model *m, size_t len) {
    if (!m) return fail(CERA_CUDA_ERR_BAD_ARG, "truncate_kv: null model");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    if (len >= m->seq_len) return CERA_CUDA_OK;
    CERA_TRY(m->rewind(len));
    m->seq_len = len;
    m->history.resize(len);
    return CERA_CUDA_OK;
}

size_t cera_cuda_kv_snapshot_bytes(const cera_cuda_model *m) { return m && m->finalized ? m->snapshot_bytes() : 0; }

int32_t cera_cuda_kv_snapshot(cera_cuda_model *m, void *out, size_t out_bytes) {
    if (!m || !out) return fail(CERA_CUDA_ERR_BAD_ARG, "kv_snapshot: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    if (!m->finalized) return fail(CERA_CUDA_ERR_STATE, "kv_snapshot: model_finalize has not been called");
    return m->snapshot(out, out_bytes);
}

int32_t cera_cuda_kv_restore(cera_cuda_model *m, const void *data, size_t bytes) {
    if (!m || !data) return fail(CERA_CUDA_ERR_BAD_ARG, "kv_restore: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    if (!m->finalized) return fail(CERA_CUDA_ERR_STATE, "kv_restore: model_finalize has not been called");
    return m->restore(data, bytes);
}

size_t cera_cuda_seq_len(const cera_cuda_model *m) { return m ? m->seq_len : 0; }
size_t cera_cuda_memory_bytes(const cera_cuda_model *m) { return m ? m->mem_bytes : 0; }
uint64_t cera_cuda_launch_count(const cera_cuda_model *m) { return m ? m->launches : 0; }

int32_t cera_cuda_last_hidden(cera_cuda_model *m, float *out) {
    if (!m || !out) return fail(CERA_CUDA_ERR_BAD_ARG, "last_hidden: null argument");
    std::lock_guard<std::mutex> lock(m->mu);
    DeviceGuard dg(m->device);
    if (!m->finalized) return fail(CERA_CUDA_ERR_STATE, "last_hidden: model not finalized");
    CERA_CUDA_TRY(cudaStreamSynchronize(m->stream));
    return check_cuda(cudaMemcpy(out, m->final_hidden, (size_t)m->hidden_size * 4, cudaMemcpyDeviceToHost), "cudaMemcpy(last_hidden)");
}

void cera_cuda_model_free(cera_cuda_model *m) { delete m; }

}  // extern "C"
