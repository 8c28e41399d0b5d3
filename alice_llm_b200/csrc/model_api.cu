// The alice_model_* entry points that are the same for every model family (include/alice_cuda.h): stepping, greedy decoding
// from a captured graph, logits, position. GpuModel of ALICE-LLM src/gpu.rs:5010-6094.
#include <vector>

#include "model_base.cuh"

namespace {

int check_room(const alice_model* m, uint32_t steps, const char* who) {
    if ((uint64_t)m->pos + steps > m->max_seq)
        return alice_fail(ALICE_E_SHAPE, "%s: position %u + %u steps exceeds max_seq_len %u", who, m->pos, steps, m->max_seq);
    return ALICE_OK;
}

int set_tokens(alice_model* m, const uint32_t* tokens, uint32_t n) {
    for (uint32_t k = 0; k < n; k++)
        if (tokens[k] >= m->vocab) return alice_fail(ALICE_E_INVALID, "alice_model: token %u >= vocab %u", tokens[k], m->vocab);
    static_assert(sizeof(uint32_t) == sizeof(int), "tokens are copied as 32-bit words");
    MCU(cudaMemcpyAsync(m->d_token, tokens, (size_t)4 * n, cudaMemcpyHostToDevice, m->e->stream));
    MCU(cudaStreamSynchronize(m->e->stream));  // the caller's array is only borrowed
    return ALICE_OK;
}

}  // namespace

extern "C" {

int32_t alice_model_destroy(alice_model* m) {
    if (!m) return ALICE_OK;
    alice_engine* e = m->e;
    cudaSetDevice(e->device);
    if (!e->dead) cudaStreamSynchronize(e->stream);
    if (m->graph_greedy) cudaGraphExecDestroy(m->graph_greedy);
    std::vector<void*> owned;
    owned.swap(m->owned);
    delete m;
    for (void* p : owned) cudaFree(p);
    alice_engine_release(e);
    return ALICE_OK;
}

int32_t alice_model_forward(alice_model* m, uint32_t token) {
    if (!m) return alice_fail(ALICE_E_INVALID, "alice_model_forward: null model");
    MCU(cudaSetDevice(m->e->device));
    int rc = check_room(m, 1, "alice_model_forward");
    if (!rc) rc = set_tokens(m, &token, 1);
    if (!rc) rc = m->enqueue_step(1, false);
    if (!rc) m->pos += 1;
    return rc;
}

int32_t alice_model_forward_batch(alice_model* m, const uint32_t* tokens, uint32_t n) {
    const char* who = "alice_model_forward_batch";
    if (!m || !tokens) return alice_fail(ALICE_E_INVALID, "%s: null argument", who);
    if (n == 0 || n > m->max_tokens()) return alice_fail(ALICE_E_SHAPE, "%s: %u tokens outside 1..%u", who, n, m->max_tokens());
    MCU(cudaSetDevice(m->e->device));
    int rc = check_room(m, n, who);
    if (!rc) rc = set_tokens(m, tokens, n);
    if (!rc) rc = m->enqueue_step(n, false);
    if (!rc) m->pos += n;
    return rc;
}

int32_t alice_model_forward_rows(alice_model* m, const uint32_t* tokens, uint32_t n, const uint32_t* rows, uint32_t nrows, float* logits) {
    const char* who = "alice_model_forward_rows";
    if (!m || !tokens || (nrows && (!rows || !logits))) return alice_fail(ALICE_E_INVALID, "%s: null argument", who);
    if (n == 0) return nrows ? alice_fail(ALICE_E_SHAPE, "%s: rows of no tokens", who) : (int)ALICE_OK;
    for (uint32_t i = 0; i < nrows; i++)
        if (rows[i] >= n || (i && rows[i] <= rows[i - 1])) return alice_fail(ALICE_E_SHAPE, "%s: rows must ascend and lie below %u", who, n);
    MCU(cudaSetDevice(m->e->device));
    int rc = check_room(m, n, who);
    uint32_t done = 0;
    std::vector<uint32_t> local;
    for (uint32_t lo = 0; lo < n && !rc;) {
        const uint32_t k = std::min(m->max_tokens(), n - lo);
        local.clear();
        while (done + local.size() < nrows && rows[done + local.size()] < lo + k) local.push_back(rows[done + local.size()] - lo);
        rc = set_tokens(m, tokens + lo, k);
        if (!rc) rc = m->enqueue_rows(k, local.data(), (uint32_t)local.size(), logits + (size_t)done * m->vocab);
        if (!rc) m->pos += k;
        done += (uint32_t)local.size();
        lo += k;
    }
    if (rc) return rc;
    return alice_sync(m->e);
}

int32_t alice_model_forward_batch_read(alice_model* m, const uint32_t* tokens, uint32_t n, float* logits) {
    const char* who = "alice_model_forward_batch_read";
    if (!m || !tokens || !logits) return alice_fail(ALICE_E_INVALID, "%s: null argument", who);
    if (n == 0 || n > m->max_tokens()) return alice_fail(ALICE_E_SHAPE, "%s: %u tokens outside 1..%u", who, n, m->max_tokens());
    std::vector<uint32_t> rows(n);
    for (uint32_t i = 0; i < n; i++) rows[i] = i;
    return alice_model_forward_rows(m, tokens, n, rows.data(), n, logits);
}

int32_t alice_model_read_logits(alice_model* m, float* logits) {
    if (!m || !logits) return alice_fail(ALICE_E_INVALID, "alice_model_read_logits: null argument");
    MCU(cudaMemcpyAsync(logits, m->logits, (size_t)m->vocab * 4, cudaMemcpyDeviceToHost, m->e->stream));
    MCU(cudaStreamSynchronize(m->e->stream));
    return alice_sync(m->e);
}

int32_t alice_model_forward_read(alice_model* m, uint32_t token, float* logits) {
    int rc = alice_model_forward(m, token);
    if (rc) return rc;
    return alice_model_read_logits(m, logits);
}

int32_t alice_model_decode_greedy(alice_model* m, uint32_t first_token, uint32_t n, uint32_t* out_tokens) {
    const char* who = "alice_model_decode_greedy";
    if (!m || (!out_tokens && n)) return alice_fail(ALICE_E_INVALID, "%s: null argument", who);
    if (n == 0) return ALICE_OK;
    MCU(cudaSetDevice(m->e->device));
    int rc = check_room(m, n, who);
    if (!rc) rc = set_tokens(m, &first_token, 1);
    if (rc) return rc;
    cudaStream_t st = m->e->stream;
    const uint32_t pos0 = m->pos;
    if (!m->graph_tried) {
        // Capture one step (every kernel reads position and token from device memory) and replay it.
        m->graph_tried = true;
        rc = m->enqueue_step(1, true);   // eager first step: also sets per-kernel attributes outside capture
        if (rc) return rc;
        m->pos += 1;
        cudaGraph_t g = nullptr;
        if (cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal) == cudaSuccess) {
            const int crc = m->enqueue_step(1, true);
            cudaError_t err = cudaStreamEndCapture(st, &g);
            if (crc == ALICE_OK && err == cudaSuccess && g) {
                if (cudaGraphInstantiate(&m->graph_greedy, g, 0) != cudaSuccess) m->graph_greedy = nullptr;
            }
            if (g) cudaGraphDestroy(g);
            cudaGetLastError();  // a failed capture only means the steps are launched one by one
        }
    }
    while (m->pos < pos0 + n) {
        if (m->graph_greedy) {
            MCU(cudaGraphLaunch(m->graph_greedy, st));
        } else {
            rc = m->enqueue_step(1, true);
            if (rc) return rc;
        }
        m->pos += 1;
    }
    static_assert(sizeof(uint32_t) == sizeof(int), "token trace is copied as 32-bit words");
    MCU(cudaMemcpyAsync(out_tokens, m->d_trace + pos0, (size_t)n * 4, cudaMemcpyDeviceToHost, st));
    MCU(cudaStreamSynchronize(st));
    return alice_sync(m->e);
}

int32_t alice_model_position(const alice_model* m, uint32_t* pos) {
    if (!m || !pos) return alice_fail(ALICE_E_INVALID, "alice_model_position: null argument");
    *pos = m->pos;
    return ALICE_OK;
}

int32_t alice_model_vocab_size(const alice_model* m, uint32_t* vocab) {
    if (!m || !vocab) return alice_fail(ALICE_E_INVALID, "alice_model_vocab_size: null argument");
    *vocab = m->vocab;
    return ALICE_OK;
}

int32_t alice_model_set_position(alice_model* m, uint32_t pos) {
    if (!m) return alice_fail(ALICE_E_INVALID, "alice_model_set_position: null model");
    if (pos > m->max_seq) return alice_fail(ALICE_E_SHAPE, "alice_model_set_position: %u > max_seq_len %u", pos, m->max_seq);
    if (!m->can_return_to(pos))
        return alice_fail(ALICE_E_UNSUPPORTED, "alice_model_set_position: the recurrent state of position %u is not kept (only reset and the present position %u can be had)", pos, m->pos);
    const int p = (int)pos;
    MCU(cudaSetDevice(m->e->device));
    MCU(cudaMemcpyAsync(m->d_pos, &p, 4, cudaMemcpyHostToDevice, m->e->stream));
    MCU(cudaStreamSynchronize(m->e->stream));
    m->pos = pos;
    return ALICE_OK;
}

int32_t alice_model_rollback_to(alice_model* m, uint32_t pos) {
    if (!m) return alice_fail(ALICE_E_INVALID, "alice_model_rollback_to: null model");
    if (pos > m->pos) return ALICE_OK;  // only ever lowers the counter (src/gpu.rs:5645-5652)
    return alice_model_set_position(m, pos);
}

int32_t alice_model_reset(alice_model* m) {
    if (!m) return alice_fail(ALICE_E_INVALID, "alice_model_reset: null model");
    MCU(cudaSetDevice(m->e->device));
    const int rc = m->clear_state();
    if (rc) return rc;
    m->pos = 0;
    return alice_model_set_position(m, 0);
}

}  // extern "C"
