// What every device-resident model shares behind the alice_model handle: position, token feed, logits, greedy trace and
// the captured decode step. A model family supplies its step and its per-sequence state (csrc/model_api.cu drives them).
#pragma once
#include <algorithm>
#include <vector>

#include "abi_internal.cuh"

struct alice_model {
    alice_engine* e = nullptr;
    uint32_t vocab = 0, max_seq = 0;
    float* logits = nullptr;
    unsigned long long* argmax_keys = nullptr;   // packed maxima left by the output head, one per tensor-parallel rank
    // device-side state: position, current tokens, tokens chosen per position
    int *d_pos = nullptr, *d_token = nullptr, *d_trace = nullptr;
    uint32_t pos = 0;                            // host mirror of *d_pos
    cudaGraphExec_t graph_greedy = nullptr;
    bool graph_tried = false;
    std::vector<void*> owned;                    // device allocations freed with the model

    virtual ~alice_model() = default;
    // Most consecutive tokens one enqueue_* call takes.
    virtual uint32_t max_tokens() const = 0;
    // Queues n consecutive tokens (read from d_token) at the current position: leaves logits and advances *d_pos. With
    // greedy_feed (n == 1) the argmax becomes the next token and is recorded in d_trace.
    virtual int enqueue_step(uint32_t n, bool greedy_feed) = 0;
    // The same n tokens with the logits of rows[0 .. nrows) (ascending, < n) copied to host_logits [nrows][vocab].
    virtual int enqueue_rows(uint32_t n, const uint32_t* rows, uint32_t nrows, float* host_logits) = 0;
    // Queues clearing of everything a sequence leaves behind.
    virtual int clear_state() = 0;
    // Whether the state after the first p tokens can be had from the present one without running them again.
    virtual bool can_return_to(uint32_t p) const { (void)p; return true; }
};

#define MCU(call)                                                       \
    do {                                                                \
        cudaError_t err__ = (call);                                     \
        if (err__ != cudaSuccess) return alice_cuda_fail(err__, #call); \
    } while (0)

template <class T>
int dev_alloc(alice_model* m, T** p, size_t n) {
    void* q = nullptr;
    cudaError_t err = cudaMalloc(&q, std::max<size_t>(n, 1) * sizeof(T));
    if (err != cudaSuccess) return alice_cuda_fail(err, "alice_model_create: cudaMalloc");
    m->owned.push_back(q);
    *p = static_cast<T*>(q);
    return ALICE_OK;
}
