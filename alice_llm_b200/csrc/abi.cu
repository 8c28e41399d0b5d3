// extern "C" surface of the quantized matvec (include/alice_cuda.h): ternary uploads, Q8_K activations, dispatch.
// The engine itself, plain weight uploads and f32 buffers are in engine.cu.
#include <cuda_runtime.h>

#include <algorithm>
#include <cstdarg>
#include <cstdio>
#include <cstring>
#include <mutex>
#include <new>
#include <string>
#include <vector>

#include "abi_internal.cuh"
#include "gemv_plan.cuh"
#include "tp.cuh"

using namespace alice;

namespace {

__device__ __forceinline__ void pdl_wait_abi() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

#define fail alice_fail
#define cuda_fail alice_cuda_fail
#define quiesce alice_quiesce
#define CU(call)                                               \
    do {                                                       \
        cudaError_t err__ = (call);                            \
        if (err__ != cudaSuccess) return cuda_fail(err__, #call); \
    } while (0)

LaunchCfg cfg_of(const alice_engine* e) { return alice_cfg_of(e); }

}  // namespace

namespace {

Q8KView view_of(const alice_q8k* q, uint32_t k) {
    auto* p = static_cast<uint8_t*>(q->base);
    Q8KView v;
    v.qs = reinterpret_cast<const int8_t*>(p + q->lay.qs_off) + (size_t)k * q->nb * 256;
    v.d = reinterpret_cast<const float*>(p + q->lay.d_off) + (size_t)k * q->nb;
    v.bsums = reinterpret_cast<const int16_t*>(p + q->lay.bsums_off) + (size_t)k * q->nb * 16;
    v.nb = q->nb;
    return v;
}

// Engine scratch grows on demand and is reused by later calls on the same stream.
int ensure_scratch(alice_engine* e, size_t bytes) {
    if (bytes <= e->scratch_bytes) return ALICE_OK;
    CU(cudaStreamSynchronize(e->stream));
    if (e->scratch) CU(cudaFree(e->scratch));
    e->scratch = nullptr; e->scratch_bytes = 0;
    CU(cudaMalloc(&e->scratch, bytes));
    e->scratch_bytes = bytes;
    return ALICE_OK;
}

int ensure_prep(alice_engine* e, size_t bytes) {
    if (bytes <= e->prep_bytes) return ALICE_OK;
    CU(cudaStreamSynchronize(e->stream));
    if (e->prep) CU(cudaFree(e->prep));
    e->prep = nullptr; e->prep_bytes = 0;
    CU(cudaMalloc(&e->prep, bytes));
    e->prep_bytes = bytes;
    return ALICE_OK;
}

int launch_rc(int rc, const char* what) {
    if (rc == ALICE_OK) return rc;
    if (rc == ALICE_E_CUDA) return fail(rc, "%s: launch failed: %s", what, cudaGetErrorString(cudaGetLastError()));
    if (rc == ALICE_E_SHAPE) return fail(rc, "%s: shape not supported by the streaming kernel", what);
    return fail(rc, "%s: error %d", what, rc);
}

}  // namespace

extern "C" {

int32_t alice_debug_expire_wait(alice_engine* e) {
    if (!e) return fail(ALICE_E_INVALID, "alice_debug_expire_wait: null engine");
    CU(cudaSetDevice(e->device));
    // scratch: [256 floats source][epoch u32][own flag u32][peer flag u32], all zero: the gate expects
    // (epoch + 1) * 1 = 1 at the own flag, which nothing raises
    int rc = ensure_scratch(e, 4096);
    if (rc) return rc;
    CU(cudaMemsetAsync(e->scratch, 0, 4096, e->stream));
    auto* base = static_cast<uint8_t*>(e->scratch);
    Publish p{};
    p.mode = PUB_VECTOR; p.n = 256; p.batch = 1; p.src = reinterpret_cast<const float*>(base);
    p.npeers = 1;
    p.epoch = reinterpret_cast<const unsigned int*>(base + 1024);
    p.wait_flag = reinterpret_cast<const unsigned int*>(base + 1028);
    p.peer_flag[0] = reinterpret_cast<unsigned int*>(base + 1032);
    p.wait_limit = e->wait_limit;
    CU(launch_publish_vector(p, e->status, e->stream, e->pdl));
    return ALICE_OK;
}

// ---- weights -------------------------------------------------------------------------------

static int upload_rows_and_scales(alice_engine* e, const std::vector<uint8_t>& host, const float* scales,
                                  WeightDesc d, alice_weights** out) {
    CU(cudaSetDevice(e->device));
    void* p = nullptr;
    void* s = nullptr;
    CU(cudaMalloc(&p, host.size() + 64));
    cudaError_t err = cudaMalloc(&s, (size_t)d.rows * sizeof(float));
    if (err == cudaSuccess) err = cudaMemcpyAsync(p, host.data(), host.size(), cudaMemcpyHostToDevice, e->stream);
    if (err == cudaSuccess) err = cudaMemsetAsync(static_cast<uint8_t*>(p) + host.size(), 0, 64, e->stream);
    if (err == cudaSuccess) err = cudaMemcpyAsync(s, scales, (size_t)d.rows * sizeof(float), cudaMemcpyHostToDevice, e->stream);
    if (err == cudaSuccess) err = cudaStreamSynchronize(e->stream);
    if (err != cudaSuccess) { cudaFree(p); if (s) cudaFree(s); return cuda_fail(err, "ternary upload"); }
    d.data = static_cast<const uint8_t*>(p);
    d.scales = static_cast<const float*>(s);
    *out = new alice_weights{e, d, p, s};
    alice_engine_retain(e);
    return ALICE_OK;
}

int32_t alice_upload_ternary(alice_engine* e, const uint8_t* pos, const uint8_t* neg, const float* scales,
                             uint32_t rows, uint32_t cols, alice_weights** out) {
    if (!e || !pos || !neg || !scales || !out) return fail(ALICE_E_INVALID, "alice_upload_ternary: null argument");
    if (rows == 0 || cols == 0) return fail(ALICE_E_SHAPE, "alice_upload_ternary: empty matrix");
    // device row = [pos plane | neg plane]; planes padded with zero bits to a whole number of 32-bit words
    const uint32_t src_pb = (cols + 7) / 8, pb = ((cols + 31) / 32) * 4;
    std::vector<uint8_t> host((size_t)rows * 2 * pb, 0);
    const uint8_t tail_mask = (cols % 8) ? (uint8_t)((1u << (cols % 8)) - 1) : 0xFF;
    for (uint32_t r = 0; r < rows; r++) {
        uint8_t* dp = host.data() + (size_t)r * 2 * pb;
        memcpy(dp, pos + (size_t)r * src_pb, src_pb);
        memcpy(dp + pb, neg + (size_t)r * src_pb, src_pb);
        dp[src_pb - 1] &= tail_mask;       // bits past num_cols are never read by the reference
        dp[pb + src_pb - 1] &= tail_mask;
    }
    WeightDesc d = {};
    d.fmt = WF_TERNARY; d.rows = rows; d.cols = cols; d.row_bytes = 2 * pb;
    return upload_rows_and_scales(e, host, scales, d, out);
}

int32_t alice_ternary_from_device(alice_engine* e, const void* rows_dptr, const float* scales_dptr, uint32_t rows,
                                  uint32_t cols, alice_weights** out) {
    if (!e || !rows_dptr || !scales_dptr || !out) return fail(ALICE_E_INVALID, "alice_ternary_from_device: null argument");
    if (rows == 0 || cols == 0) return fail(ALICE_E_SHAPE, "alice_ternary_from_device: empty matrix");
    if ((uintptr_t)rows_dptr & 15) return fail(ALICE_E_INVALID, "alice_ternary_from_device: pointer not 16-byte aligned");
    const uint32_t pb = ((cols + 31) / 32) * 4;
    if (((size_t)rows * 2 * pb) & 15)
        return fail(ALICE_E_SHAPE, "alice_ternary_from_device: rows * row bytes (%zu) must be a multiple of 16", (size_t)rows * 2 * pb);
    WeightDesc d = {};
    d.fmt = WF_TERNARY; d.rows = rows; d.cols = cols; d.row_bytes = 2 * pb;
    d.data = static_cast<const uint8_t*>(rows_dptr);
    d.scales = scales_dptr;
    *out = new alice_weights{e, d, nullptr, nullptr};
    alice_engine_retain(e);
    return ALICE_OK;
}

int32_t alice_upload_sparse_ternary(alice_engine* e, const uint8_t* packed, const float* scales, uint32_t rows,
                                    uint32_t cols, alice_weights** out) {
    if (!e || !packed || !scales || !out) return fail(ALICE_E_INVALID, "alice_upload_sparse_ternary: null argument");
    if (rows == 0 || cols == 0) return fail(ALICE_E_SHAPE, "alice_upload_sparse_ternary: empty matrix");
    const uint32_t rb = ((cols + 15) / 16) * 4;
    std::vector<uint8_t> host(packed, packed + (size_t)rows * rb);
    WeightDesc d = {};
    d.fmt = WF_SPARSE_TERNARY; d.rows = rows; d.cols = cols; d.row_bytes = rb;
    return upload_rows_and_scales(e, host, scales, d, out);
}

// ---- Q8_K activations ----------------------------------------------------------------------

int32_t alice_q8k_alloc(alice_engine* e, uint32_t cols, uint32_t batch, alice_q8k** out) {
    if (!e || !out) return fail(ALICE_E_INVALID, "alice_q8k_alloc: null argument");
    if (cols == 0 || cols % 256 != 0) return fail(ALICE_E_SHAPE, "alice_q8k_alloc: cols %u is not a multiple of 256", cols);
    if (batch == 0) return fail(ALICE_E_SHAPE, "alice_q8k_alloc: batch 0");
    CU(cudaSetDevice(e->device));
    auto* q = new alice_q8k{e, nullptr, cols, batch, cols / 256, Q8KLayout::make(cols / 256, batch)};
    cudaError_t err = cudaMalloc(&q->base, q->lay.total);
    if (err != cudaSuccess) { delete q; return cuda_fail(err, "alice_q8k_alloc"); }
    alice_engine_retain(e);
    *out = q;
    return ALICE_OK;
}

int32_t alice_quantize_q8k(alice_engine* e, const alice_buf* x, alice_q8k* q) {
    if (!e || !x || !q) return fail(ALICE_E_INVALID, "alice_quantize_q8k: null argument");
    if (x->len < (size_t)q->cols * q->batch)
        return fail(ALICE_E_SHAPE, "alice_quantize_q8k: input has %zu floats, need %zu", x->len, (size_t)q->cols * q->batch);
    launch_quantize_q8k(x->p, q->cols, q->batch, q->base, e->stream, e->pdl);
    CU(cudaGetLastError());
    return ALICE_OK;
}

int32_t alice_q8k_read(alice_engine* e, const alice_q8k* q, float* d, int8_t* qs, int16_t* bsums) {
    if (!e || !q || !d || !qs || !bsums) return fail(ALICE_E_INVALID, "alice_q8k_read: null argument");
    const size_t n = (size_t)q->batch * q->nb;
    auto* p = static_cast<const uint8_t*>(q->base);
    CU(cudaMemcpyAsync(qs, p + q->lay.qs_off, n * 256, cudaMemcpyDeviceToHost, e->stream));
    CU(cudaMemcpyAsync(d, p + q->lay.d_off, n * 4, cudaMemcpyDeviceToHost, e->stream));
    CU(cudaMemcpyAsync(bsums, p + q->lay.bsums_off, n * 32, cudaMemcpyDeviceToHost, e->stream));
    CU(cudaStreamSynchronize(e->stream));
    return ALICE_OK;
}

int32_t alice_q8k_upload(alice_engine* e, const float* d, const int8_t* qs, const int16_t* bsums, uint32_t cols,
                         uint32_t batch, alice_q8k** out) {
    if (!d || !qs || !bsums) return fail(ALICE_E_INVALID, "alice_q8k_upload: null argument");
    int rc = alice_q8k_alloc(e, cols, batch, out);
    if (rc) return rc;
    alice_q8k* q = *out;
    const size_t n = (size_t)batch * q->nb;
    auto* p = static_cast<uint8_t*>(q->base);
    cudaError_t err = cudaMemcpyAsync(p + q->lay.qs_off, qs, n * 256, cudaMemcpyHostToDevice, e->stream);
    if (err == cudaSuccess) err = cudaMemcpyAsync(p + q->lay.d_off, d, n * 4, cudaMemcpyHostToDevice, e->stream);
    if (err == cudaSuccess) err = cudaMemcpyAsync(p + q->lay.bsums_off, bsums, n * 32, cudaMemcpyHostToDevice, e->stream);
    if (err == cudaSuccess) err = cudaStreamSynchronize(e->stream);
    if (err != cudaSuccess) { alice_q8k_free(q); *out = nullptr; return cuda_fail(err, "alice_q8k_upload"); }
    return ALICE_OK;
}

int32_t alice_q8k_free(alice_q8k* q) {
    if (!q) return ALICE_OK;
    quiesce(q->e);
    cudaFree(q->base);
    alice_engine_release(q->e);
    delete q;
    return ALICE_OK;
}

// ---- the hot path --------------------------------------------------------------------------

Q8KView view_at(void* base, uint32_t nb, uint32_t batch) {
    const Q8KLayout l = Q8KLayout::make(nb, batch);
    auto* p = static_cast<uint8_t*>(base);
    Q8KView v;
    v.qs = reinterpret_cast<const int8_t*>(p + l.qs_off);
    v.d = reinterpret_cast<const float*>(p + l.d_off);
    v.bsums = reinterpret_cast<const int16_t*>(p + l.bsums_off);
    v.nb = nb;
    return v;
}

// One matvec / fused SwiGLU over `batch` prepared input vectors.
static int run_gemv(alice_engine* e, const alice_weights* w0, const alice_weights* w1, const Q8KView* q8, const float* xf,
                    float* y, uint32_t batch, const char* who, bool may_alloc = true) {
    GemvOp op;
    const WeightFormat f = w0->d.fmt;
    if (f == WF_Q1_0 || f == WF_Q2_0 || f == WF_TERNARY || f == WF_SPARSE_TERNARY) {
        // room for the activation digit table, prepared once ahead of the matvec (csrc/gemv_mma.cuh)
        if (may_alloc) { const int rc = ensure_prep(e, mma_prep_bytes(w0->d.cols)); if (rc) return rc; }
        op.prep = e->prep; op.prep_bytes = e->prep_bytes;
    }
    op.w[0] = &w0->d; op.up = w1 ? &w1->d : nullptr;
    op.q8 = q8; op.x = xf; op.y = y; op.batch = batch;
    op.wait_limit = e->wait_limit;
    return launch_rc(launch_stream_gemv_op(op, cfg_of(e)), who);
}

static int check_pair(const alice_weights* g, const alice_weights* u, const char* who) {
    if (g->d.fmt != u->d.fmt || g->d.rows != u->d.rows || g->d.cols != u->d.cols)
        return fail(ALICE_E_SHAPE, "%s: gate and up differ in format or shape", who);
    return ALICE_OK;
}

// f32 input of a matvec. K-quant weights want it as Q8_K blocks (q4k_matvec = quantize_row_q8_k + q4k_matvec_preq,
// src/gguf.rs:3600-3603): a small quantizer kernel runs ahead of the matvec, which is launched as its programmatic
// dependent - its CTAs become resident and stream weights while the blocks are being written. (Measured on the FFN
// block at 8B shapes: 31.6 us per block this way, 35.5 us with the quantization done inside the matvec kernels.)
static int matvec_common(alice_engine* e, const alice_weights* w0, const alice_weights* w1, const alice_buf* x,
                         alice_buf* y, uint32_t batch, const char* who) {
    if (!e || !w0 || !x || !y) return fail(ALICE_E_INVALID, "%s: null argument", who);
    if (batch == 0 || batch > 8) return fail(ALICE_E_SHAPE, "%s: batch %u outside 1..8", who, batch);
    if (w1) { int rc = check_pair(w0, w1, who); if (rc) return rc; }
    const WeightDesc& d = w0->d;
    if (x->len < (size_t)batch * d.cols) return fail(ALICE_E_SHAPE, "%s: input has %zu floats, need %zu", who, x->len, (size_t)batch * d.cols);
    if (y->len < (size_t)batch * d.rows) return fail(ALICE_E_SHAPE, "%s: output has %zu floats, need %zu", who, y->len, (size_t)batch * d.rows);
    CU(cudaSetDevice(e->device));
    if (!format_uses_q8k(d.fmt)) return run_gemv(e, w0, w1, nullptr, x->p, y->p, batch, who);
    if ((uintptr_t)x->p & 15) return fail(ALICE_E_INVALID, "%s: input vector must be 16-byte aligned", who);
    const uint32_t nb = d.cols / 256;
    int rc = ensure_scratch(e, Q8KLayout::make(nb, batch).total);
    if (rc) return rc;
    launch_quantize_q8k(x->p, d.cols, batch, e->scratch, e->stream, e->pdl);
    CU(cudaGetLastError());
    const Q8KView v = view_at(e->scratch, nb, batch);
    return run_gemv(e, w0, w1, &v, nullptr, y->p, batch, who);
}

static int preq_common(alice_engine* e, const alice_weights* w0, const alice_weights* w1, const alice_q8k* q,
                       alice_buf* y, const char* who) {
    if (!e || !w0 || !q || !y) return fail(ALICE_E_INVALID, "%s: null argument", who);
    if (w1) { int rc = check_pair(w0, w1, who); if (rc) return rc; }
    const WeightDesc& d = w0->d;
    if (q->cols != d.cols) return fail(ALICE_E_SHAPE, "%s: Q8_K input has %u columns, weights %u", who, q->cols, d.cols);
    if (q->batch > 8) return fail(ALICE_E_SHAPE, "%s: batch %u outside 1..8", who, q->batch);
    if (y->len < (size_t)q->batch * d.rows) return fail(ALICE_E_SHAPE, "%s: output too small", who);
    CU(cudaSetDevice(e->device));
    if (format_uses_q8k(d.fmt)) {
        const Q8KView v = view_of(q, 0);
        return run_gemv(e, w0, w1, &v, nullptr, y->p, q->batch, who);
    }
    if (d.fmt == WF_Q1_0 || d.fmt == WF_Q2_0) {
        const size_t total = (size_t)q->batch * d.cols;
        int rc = ensure_scratch(e, total * sizeof(float));
        if (rc) return rc;
        launch_q8k_to_f32(view_of(q, 0), total, static_cast<float*>(e->scratch), e->stream);
        return run_gemv(e, w0, w1, nullptr, static_cast<float*>(e->scratch), y->p, q->batch, who);
    }
    // quantized_matvec_preq panics for every other type (src/gguf.rs:4606)
    return fail(ALICE_E_UNSUPPORTED, "%s: pre-quantized input only for Q4_K/Q5_K/Q6_K/Q1_0/Q2_0", who);
}

int32_t alice_matvec(alice_engine* e, const alice_weights* w, const alice_buf* x, alice_buf* y, uint32_t batch) {
    return matvec_common(e, w, nullptr, x, y, batch, "alice_matvec");
}

int32_t alice_matvec_preq(alice_engine* e, const alice_weights* w, const alice_q8k* q, alice_buf* y) {
    return preq_common(e, w, nullptr, q, y, "alice_matvec_preq");
}

int32_t alice_swiglu(alice_engine* e, const alice_weights* gate, const alice_weights* up, const alice_buf* x,
                     alice_buf* y, uint32_t batch) {
    if (!up) return fail(ALICE_E_INVALID, "alice_swiglu: null argument");
    return matvec_common(e, gate, up, x, y, batch, "alice_swiglu");
}

int32_t alice_swiglu_preq(alice_engine* e, const alice_weights* gate, const alice_weights* up, const alice_q8k* q,
                          alice_buf* y) {
    if (!up) return fail(ALICE_E_INVALID, "alice_swiglu_preq: null argument");
    return preq_common(e, gate, up, q, y, "alice_swiglu_preq");
}

int32_t alice_plan_query(alice_engine* e, const alice_weights* w, int32_t swiglu, int32_t preq, uint32_t* out, uint32_t n_out) {
    if (!e || !w || !out || n_out < 10) return fail(ALICE_E_INVALID, "alice_plan_query: null argument or fewer than 10 outputs");
    GemvOp op;
    op.w[0] = &w->d;
    if (swiglu) op.up = &w->d;
    alignas(16) static float dummy[4];
    Q8KView v{};
    (void)preq;     // the input always reaches the kernel prepared; the plan does not depend on who prepared it
    if (format_uses_q8k(w->d.fmt)) { v.qs = reinterpret_cast<const int8_t*>(dummy); v.nb = w->d.cols / 256; op.q8 = &v; }
    else op.x = dummy;
    op.y = dummy;   // planning never dereferences the vectors
    StreamPlan pl;
    const int rc = plan_stream_gemv(op, cfg_of(e), pl);
    if (rc) return launch_rc(rc, "alice_plan_query");
    const StreamArgs& a = pl.args;
    out[0] = pl.grid; out[1] = a.P; out[2] = a.slots; out[3] = a.rps; out[4] = a.groups; out[5] = a.nstages;
    out[6] = pl.kl; out[7] = pl.mma ? 1u : 0u; out[8] = pl.ksplit; out[9] = pl.ctas_per_sm;
    return ALICE_OK;
}

int32_t alice_batch_plan(alice_engine* e, const alice_weights* w, int32_t swiglu, uint32_t batch, uint32_t* launches, uint32_t* weight_passes) {
    if (!e || !w || !launches || !weight_passes) return fail(ALICE_E_INVALID, "alice_batch_plan: null argument");
    if (batch == 0 || batch > 8) return fail(ALICE_E_SHAPE, "alice_batch_plan: batch %u outside 1..8", batch);
    GemvOp op;
    op.w[0] = &w->d;
    if (swiglu) op.up = &w->d;
    alignas(16) static float dummy[4];
    Q8KView v{};
    if (format_uses_q8k(w->d.fmt)) { v.qs = reinterpret_cast<const int8_t*>(dummy); v.d = dummy; v.bsums = reinterpret_cast<const int16_t*>(dummy); v.nb = w->d.cols / 256; op.q8 = &v; }
    else op.x = dummy;
    op.y = dummy; op.batch = batch;
    return launch_rc(batch_plan(op, cfg_of(e), launches, weight_passes), "alice_batch_plan");
}

int32_t alice_dequantize(alice_engine* e, const alice_weights* w, alice_buf* out) {
    if (!e || !w || !out) return fail(ALICE_E_INVALID, "alice_dequantize: null argument");
    if (out->len < (size_t)w->d.rows * w->d.cols) return fail(ALICE_E_SHAPE, "alice_dequantize: output too small");
    CU(cudaSetDevice(e->device));
    return launch_rc(launch_dequantize(w->d, out->p, e->stream), "alice_dequantize");
}

// ---- host-pointer convenience --------------------------------------------------------------

static alice_engine* g_host_engine = nullptr;
static std::mutex g_host_mu;

static int host_engine(alice_engine** out) {
    if (!g_host_engine) {
        int rc = alice_engine_create(0, &g_host_engine);
        if (rc) return rc;
    }
    *out = g_host_engine;
    return ALICE_OK;
}

int32_t alice_matvec_host(uint32_t type, const uint8_t* data, size_t nbytes, uint32_t rows, uint32_t cols,
                          const float* x, float* y) {
    if (!data || !x || !y) return fail(ALICE_E_INVALID, "alice_matvec_host: null argument");
    std::lock_guard<std::mutex> lk(g_host_mu);
    alice_engine* e;
    int rc = host_engine(&e);
    if (rc) return rc;
    alice_weights* w = nullptr;
    alice_buf *bx = nullptr, *by = nullptr;
    rc = alice_upload_weights(e, data, nbytes, type, rows, cols, &w);
    if (!rc) rc = alice_buf_upload_f32(e, x, cols, &bx);
    if (!rc) rc = alice_buf_alloc_f32(e, rows, &by);
    if (!rc) rc = alice_matvec(e, w, bx, by, 1);
    if (!rc) rc = alice_buf_read_f32(e, by, y, rows);
    if (!rc) rc = alice_sync(e);
    alice_buf_free(by); alice_buf_free(bx); alice_weights_free(w);
    return rc;
}

int32_t alice_dequantize_host(uint32_t type, const uint8_t* data, size_t nbytes, float* out, size_t n_out) {
    if (!data || !out) return fail(ALICE_E_INVALID, "alice_dequantize_host: null argument");
    const uint32_t be = ggml_block_elems((WeightFormat)type);
    if (be == 0) return fail(ALICE_E_UNSUPPORTED, "alice_dequantize_host: unsupported quantization type %u", type);
    if (n_out == 0 || n_out % be != 0 || n_out > 0xFFFFFFFFu)
        return fail(ALICE_E_SHAPE, "alice_dequantize_host: %zu outputs is not a whole number of blocks", n_out);
    std::lock_guard<std::mutex> lk(g_host_mu);
    alice_engine* e;
    int rc = host_engine(&e);
    if (rc) return rc;
    alice_weights* w = nullptr;
    alice_buf* bo = nullptr;
    rc = alice_upload_weights(e, data, nbytes, type, 1, (uint32_t)n_out, &w);
    if (!rc) rc = alice_buf_alloc_f32(e, n_out, &bo);
    if (!rc) rc = alice_dequantize(e, w, bo);
    if (!rc) rc = alice_buf_read_f32(e, bo, out, n_out);
    alice_buf_free(bo); alice_weights_free(w);
    return rc;
}

// ---- pre-quantized Q1_0 / Q2_0 matvec without any allocation -------------------------------------
//
// alice_matvec_preq turns the Q8_K blocks back into f32 (src/gguf.rs:4593-4605) in a scratch
// buffer that the engine obtains with cudaMalloc and grows on demand. Some callers must not reach
// the allocator at all: a serving process that has handed every byte of HBM to its own pool
// (KV-cache arena, a framework's caching allocator) so that cudaMalloc fails; or a decode thread
// that cannot afford cudaMalloc / cudaFree because both synchronise the whole device. For them the
// variant below keeps the f32 scratch in a fixed array that is part of the library image: every
// GPU that loads the library holds ALICE_NOALLOC_MAX_FLOATS * 4 bytes (256 KiB) until the process
// exits.

static __device__ __align__(256) float g_noalloc_scratch[ALICE_NOALLOC_MAX_FLOATS];

// In host code `g_noalloc_scratch` is only a handle for the runtime, not a device address; the
// address of each device's copy is looked up once, with that device current, and cached here.
static float* g_noalloc_ptr[64] = {};
static std::mutex g_noalloc_mu;

static __global__ void q8k_to_f32_noalloc_kernel(Q8KView q, uint32_t total) {
    pdl_wait_abi();
    for (uint32_t i = blockIdx.x * blockDim.x + threadIdx.x; i < total; i += gridDim.x * blockDim.x)
        g_noalloc_scratch[i] = __fmul_rn(q.d[i >> 8], (float)q.qs[i]);
}

static int noalloc_scratch_for(alice_engine* e, float** out) {
    if (e->device < 0 || e->device >= 64) return fail(ALICE_E_INVALID, "alice_matvec_preq_noalloc: device index %d", e->device);
    std::lock_guard<std::mutex> lk(g_noalloc_mu);
    if (!g_noalloc_ptr[e->device]) {
        void* p = nullptr;
        cudaError_t err = cudaGetSymbolAddress(&p, g_noalloc_scratch);  // current device = e->device (set by the caller)
        if (err != cudaSuccess || !p) return cuda_fail(err, "alice_matvec_preq_noalloc: cudaGetSymbolAddress");
        g_noalloc_ptr[e->device] = static_cast<float*>(p);
    }
    *out = g_noalloc_ptr[e->device];
    return ALICE_OK;
}

int32_t alice_matvec_preq_noalloc(alice_engine* e, const alice_weights* w, const alice_q8k* q, alice_buf* y) {
    const char* who = "alice_matvec_preq_noalloc";
    if (!e || !w || !q || !y) return fail(ALICE_E_INVALID, "%s: null argument", who);
    const WeightDesc& d = w->d;
    if (d.fmt != WF_Q1_0 && d.fmt != WF_Q2_0)
        return fail(ALICE_E_UNSUPPORTED, "%s: only Q1_0 / Q2_0 weights need the f32 scratch; use alice_matvec_preq", who);
    if (q->cols != d.cols) return fail(ALICE_E_SHAPE, "%s: Q8_K input has %u columns, weights %u", who, q->cols, d.cols);
    if (q->batch == 0 || q->batch > 8) return fail(ALICE_E_SHAPE, "%s: batch %u outside 1..8", who, q->batch);
    const size_t total = (size_t)q->batch * d.cols;
    if (total > (size_t)ALICE_NOALLOC_MAX_FLOATS)
        return fail(ALICE_E_SHAPE, "%s: batch * cols = %zu floats exceeds the fixed scratch of %d floats", who, total,
                    (int)ALICE_NOALLOC_MAX_FLOATS);
    if (y->len < (size_t)q->batch * d.rows) return fail(ALICE_E_SHAPE, "%s: output too small", who);
    CU(cudaSetDevice(e->device));
    float* scratch = nullptr;
    int rc = noalloc_scratch_for(e, &scratch);
    if (rc) return rc;
    // Every element the matvec reads is rewritten first, so nothing has to be cleared between calls.
    const unsigned blocks = (unsigned)std::min<size_t>((total + 255) / 256, 148 * 8);
    q8k_to_f32_noalloc_kernel<<<blocks, 256, 0, e->stream>>>(view_of(q, 0), (uint32_t)total);
    CU(cudaGetLastError());
    return run_gemv(e, w, nullptr, nullptr, scratch, y->p, q->batch, who, false);   // never allocates
}

}  // extern "C"
