// The part of the C ABI every model family needs: errors, the engine, plain weight uploads, f32 buffers.
#include <cuda_runtime.h>

#include <algorithm>
#include <cstdarg>
#include <cstdio>
#include <new>
#include <string>

#include "abi_internal.cuh"
#include "tp.cuh"

using namespace alice;

namespace {
thread_local std::string g_err;
}

int alice_fail(int code, const char* fmt, ...) {
    char buf[512];
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(buf, sizeof buf, fmt, ap);
    va_end(ap);
    g_err = buf;
    return code;
}
int alice_cuda_fail(cudaError_t err, const char* what) {
    return alice_fail(err == cudaErrorMemoryAllocation ? ALICE_E_NOMEM : ALICE_E_CUDA, "%s: %s", what, cudaGetErrorString(err));
}

#define fail alice_fail
#define cuda_fail alice_cuda_fail
#define quiesce alice_quiesce
#define CU(call)                                               \
    do {                                                       \
        cudaError_t err__ = (call);                            \
        if (err__ != cudaSuccess) return cuda_fail(err__, #call); \
    } while (0)

void alice_engine_retain(alice_engine* e) { e->refs++; }
void alice_engine_release(alice_engine* e) {
    if (--e->refs == 0) delete e;
}
// Before a handle frees device memory the engine's queued work must be done - unless the engine is already gone
// (its destroy synchronised the stream).
void alice_quiesce(alice_engine* e) {
    cudaSetDevice(e->device);
    if (!e->dead) cudaStreamSynchronize(e->stream);
}

LaunchCfg alice_cfg_of(const alice_engine* e) {
    LaunchCfg c;
    c.stream = e->stream; c.num_sms = e->num_sms; c.status = e->status; c.pdl = e->pdl;
    c.force_rps = e->force_rps; c.force_stages = e->force_stages;
    return c;
}

namespace alice {
uint32_t ggml_block_bytes(WeightFormat f) {
    switch (f) {
        case WF_Q8_0: return 34; case WF_Q4_K: return 144; case WF_Q5_K: return 176;
        case WF_Q6_K: return 210; case WF_Q1_0: return 18; case WF_Q2_0: return 34;
        case WF_BF16: return 2;
        default: return 0;
    }
}
uint32_t ggml_block_elems(WeightFormat f) {
    switch (f) {
        case WF_Q8_0: return 32;
        case WF_Q4_K: case WF_Q5_K: case WF_Q6_K: return 256;
        case WF_Q1_0: case WF_Q2_0: return 128;
        case WF_BF16: return 1;
        default: return 0;
    }
}
uint32_t ggml_row_bytes(WeightFormat f, uint32_t cols) {
    const uint32_t e = ggml_block_elems(f);
    if (e == 0 || cols == 0 || cols % e != 0) return 0;
    return cols / e * ggml_block_bytes(f);
}

}  // namespace alice

namespace {
bool known_ggml(uint32_t t) { return ggml_block_bytes((WeightFormat)t) != 0; }

}  // namespace

extern "C" {

const char* alice_last_error(void) { return g_err.c_str(); }

uint32_t alice_type_block_bytes(uint32_t t) { return ggml_block_bytes((WeightFormat)t); }
uint32_t alice_type_block_elems(uint32_t t) { return ggml_block_elems((WeightFormat)t); }

int32_t alice_engine_create(int32_t device, alice_engine** out) {
    if (!out) return fail(ALICE_E_INVALID, "alice_engine_create: out is null");
    *out = nullptr;
    int n = 0;
    cudaError_t err = cudaGetDeviceCount(&n);
    if (err != cudaSuccess || n == 0)
        return fail(ALICE_E_CUDA, "alice_engine_create: no CUDA device (%s); this library has no CPU path",
                    cudaGetErrorString(err));
    if (device < 0 || device >= n) return fail(ALICE_E_INVALID, "alice_engine_create: device %d of %d", device, n);
    CU(cudaSetDevice(device));
    cudaDeviceProp prop;
    CU(cudaGetDeviceProperties(&prop, device));
    if (prop.major < 10)
        return fail(ALICE_E_UNSUPPORTED, "alice_engine_create: device is sm_%d%d; kernels are built for sm_100a",
                    prop.major, prop.minor);
    auto* e = new (std::nothrow) alice_engine();
    if (!e) return fail(ALICE_E_NOMEM, "alice_engine_create: host allocation failed");
    e->device = device;
    e->num_sms = prop.multiProcessorCount;
    err = cudaStreamCreateWithFlags(&e->stream, cudaStreamNonBlocking);
    if (err != cudaSuccess) { delete e; return cuda_fail(err, "cudaStreamCreate"); }
    e->own_stream = true;
    err = cudaMalloc(&e->status, sizeof(int));
    if (err == cudaSuccess) err = cudaMemset(e->status, 0, sizeof(int));
    if (err == cudaSuccess) err = cudaMallocHost(reinterpret_cast<void**>(&e->status_host), sizeof(int));
    if (err != cudaSuccess) {
        if (e->status) cudaFree(e->status);
        if (e->status_host) cudaFreeHost(e->status_host);
        cudaStreamDestroy(e->stream); delete e;
        return cuda_fail(err, "status word");
    }
    *out = e;
    return ALICE_OK;
}

int32_t alice_engine_destroy(alice_engine* e) {
    if (!e || e->dead) return ALICE_OK;
    cudaSetDevice(e->device);
    cudaStreamSynchronize(e->stream);
    alice::tp_release(e);
    if (e->scratch) cudaFree(e->scratch);
    if (e->prep) cudaFree(e->prep);
    if (e->status) cudaFree(e->status);
    if (e->status_host) cudaFreeHost(e->status_host);
    if (e->own_stream) cudaStreamDestroy(e->stream);
    e->scratch = e->prep = nullptr; e->status = nullptr; e->status_host = nullptr; e->stream = nullptr;
    e->dead = true;               // handles created on this engine may outlive it: they only free their own memory
    alice_engine_release(e);
    return ALICE_OK;
}

int32_t alice_engine_set_stream(alice_engine* e, void* s) {
    if (!e) return fail(ALICE_E_INVALID, "alice_engine_set_stream: null engine");
    CU(cudaStreamSynchronize(e->stream));
    if (e->own_stream) { cudaStreamDestroy(e->stream); e->own_stream = false; }
    e->stream = static_cast<cudaStream_t>(s);
    return ALICE_OK;
}

int32_t alice_engine_set_pdl(alice_engine* e, int32_t on) {
    if (!e) return fail(ALICE_E_INVALID, "alice_engine_set_pdl: null engine");
    e->pdl = on != 0;
    return ALICE_OK;
}

int32_t alice_engine_set_tuning(alice_engine* e, int32_t rps, int32_t stages) {
    if (!e) return fail(ALICE_E_INVALID, "alice_engine_set_tuning: null engine");
    e->force_rps = rps; e->force_stages = stages;
    return ALICE_OK;
}

int32_t alice_engine_set_wait_limit(alice_engine* e, uint64_t sm_cycles) {
    if (!e) return fail(ALICE_E_INVALID, "alice_engine_set_wait_limit: null engine");
    e->wait_limit = (long long)std::min<uint64_t>(sm_cycles, (uint64_t)1 << 40);
    return ALICE_OK;
}

int32_t alice_sync(alice_engine* e) {
    if (!e) return fail(ALICE_E_INVALID, "alice_sync: null engine");
    CU(cudaSetDevice(e->device));
    // the status word rides the same wait: its copy to pinned host memory is queued behind the work
    CU(cudaMemcpyAsync(e->status_host, e->status, sizeof(int), cudaMemcpyDeviceToHost, e->stream));
    CU(cudaStreamSynchronize(e->stream));
    const int st = *e->status_host;
    if (st != 0) {
        cudaMemset(e->status, 0, sizeof(int));
        static const char* const what[] = {"?", "unspecified wait", "weights did not land in shared memory", "partial sums of a row", "stage release",
                                           "grid barrier", "rows from a tensor-parallel peer", "operands or accumulators of a tensor-core product", "a tile of cached keys and values", "operands or weights of tensor-core attention"};
        const int code = st & 0xff;
        return fail(ALICE_E_KERNEL, "alice_sync: a kernel wait ran out of its cycle budget (status %d: %s); results of the queued work are void",
                    st, code >= 1 && code <= 9 ? what[code] : what[0]);
    }
    return ALICE_OK;
}

// ---- weights -------------------------------------------------------------------------------

static int make_ggml_desc(const char* who, size_t nbytes, uint32_t type, uint32_t rows, uint32_t cols, WeightDesc& d) {
    if (!known_ggml(type)) return fail(ALICE_E_UNSUPPORTED, "%s: unsupported quantization type %u", who, type);
    const uint32_t rb = ggml_row_bytes((WeightFormat)type, cols);
    if (rows == 0 || rb == 0)
        return fail(ALICE_E_SHAPE, "%s: cols %u is not a whole number of %u-element blocks (rows %u)", who, cols,
                    ggml_block_elems((WeightFormat)type), rows);
    if ((size_t)rows * rb != nbytes)
        return fail(ALICE_E_SHAPE, "%s: %zu bytes given, %u x %u needs %zu", who, nbytes, rows, cols, (size_t)rows * rb);
    d = WeightDesc{};
    d.fmt = (WeightFormat)type; d.rows = rows; d.cols = cols; d.row_bytes = rb;
    return ALICE_OK;
}

int32_t alice_upload_weights(alice_engine* e, const uint8_t* data, size_t nbytes, uint32_t type, uint32_t rows,
                             uint32_t cols, alice_weights** out) {
    if (!e || !data || !out) return fail(ALICE_E_INVALID, "alice_upload_weights: null argument");
    WeightDesc d;
    int rc = make_ggml_desc("alice_upload_weights", nbytes, type, rows, cols, d);
    if (rc) return rc;
    CU(cudaSetDevice(e->device));
    void* p = nullptr;
    CU(cudaMalloc(&p, nbytes + 64));  // tail slack: bulk copies round their end up to 16 bytes
    cudaError_t err = cudaMemcpyAsync(p, data, nbytes, cudaMemcpyHostToDevice, e->stream);
    if (err == cudaSuccess) err = cudaMemsetAsync(static_cast<uint8_t*>(p) + nbytes, 0, 64, e->stream);
    if (err == cudaSuccess) err = cudaStreamSynchronize(e->stream);  // the host slice is only borrowed
    if (err != cudaSuccess) { cudaFree(p); return cuda_fail(err, "alice_upload_weights copy"); }
    d.data = static_cast<const uint8_t*>(p);
    *out = new alice_weights{e, d, p, nullptr};
    alice_engine_retain(e);
    return ALICE_OK;
}

int32_t alice_weights_from_device(alice_engine* e, const void* dptr, size_t nbytes, uint32_t type, uint32_t rows,
                                  uint32_t cols, alice_weights** out) {
    if (!e || !dptr || !out) return fail(ALICE_E_INVALID, "alice_weights_from_device: null argument");
    if ((uintptr_t)dptr & 15) return fail(ALICE_E_INVALID, "alice_weights_from_device: pointer not 16-byte aligned");
    WeightDesc d;
    int rc = make_ggml_desc("alice_weights_from_device", nbytes, type, rows, cols, d);
    if (rc) return rc;
    if (nbytes & 15)
        return fail(ALICE_E_SHAPE, "alice_weights_from_device: byte size %zu must be a multiple of 16", nbytes);
    d.data = static_cast<const uint8_t*>(dptr);
    *out = new alice_weights{e, d, nullptr, nullptr};
    alice_engine_retain(e);
    return ALICE_OK;
}

int32_t alice_weights_free(alice_weights* w) {
    if (!w) return ALICE_OK;
    if (w->owned_data || w->owned_scales) quiesce(w->e);
    if (w->owned_data) cudaFree(w->owned_data);
    if (w->owned_scales) cudaFree(w->owned_scales);
    alice_engine_release(w->e);
    delete w;
    return ALICE_OK;
}

// ---- f32 buffers ---------------------------------------------------------------------------

int32_t alice_buf_alloc_f32(alice_engine* e, size_t len, alice_buf** out) {
    if (!e || !out) return fail(ALICE_E_INVALID, "alice_buf_alloc_f32: null argument");
    CU(cudaSetDevice(e->device));
    void* p = nullptr;
    CU(cudaMalloc(&p, std::max<size_t>(len, 1) * sizeof(float)));
    cudaError_t err = cudaMemsetAsync(p, 0, std::max<size_t>(len, 1) * sizeof(float), e->stream);
    if (err != cudaSuccess) { cudaFree(p); return cuda_fail(err, "alice_buf_alloc_f32 memset"); }
    *out = new alice_buf{e, static_cast<float*>(p), len, true};
    alice_engine_retain(e);
    return ALICE_OK;
}

int32_t alice_buf_write_f32(alice_engine* e, alice_buf* b, const float* data, size_t len) {
    if (!e || !b || (!data && len)) return fail(ALICE_E_INVALID, "alice_buf_write_f32: null argument");
    if (len > b->len) return fail(ALICE_E_SHAPE, "alice_buf_write_f32: %zu floats into a buffer of %zu", len, b->len);
    CU(cudaMemcpyAsync(b->p, data, len * sizeof(float), cudaMemcpyHostToDevice, e->stream));
    CU(cudaStreamSynchronize(e->stream));  // the host slice is only borrowed for the call
    return ALICE_OK;
}

int32_t alice_buf_write_f32_async(alice_engine* e, alice_buf* b, const float* data, size_t len) {
    if (!e || !b || (!data && len)) return fail(ALICE_E_INVALID, "alice_buf_write_f32_async: null argument");
    if (len > b->len) return fail(ALICE_E_SHAPE, "alice_buf_write_f32_async: %zu floats into a buffer of %zu", len, b->len);
    CU(cudaMemcpyAsync(b->p, data, len * sizeof(float), cudaMemcpyHostToDevice, e->stream));
    return ALICE_OK;
}

int32_t alice_buf_read_f32_async(alice_engine* e, const alice_buf* b, float* out, size_t len) {
    if (!e || !b || (!out && len)) return fail(ALICE_E_INVALID, "alice_buf_read_f32_async: null argument");
    if (len > b->len) return fail(ALICE_E_SHAPE, "alice_buf_read_f32_async: %zu floats from a buffer of %zu", len, b->len);
    CU(cudaMemcpyAsync(out, b->p, len * sizeof(float), cudaMemcpyDeviceToHost, e->stream));
    return ALICE_OK;
}

int32_t alice_buf_upload_f32(alice_engine* e, const float* data, size_t len, alice_buf** out) {
    int rc = alice_buf_alloc_f32(e, len, out);
    if (rc) return rc;
    rc = alice_buf_write_f32(e, *out, data, len);
    if (rc) { alice_buf_free(*out); *out = nullptr; }
    return rc;
}

int32_t alice_buf_read_f32(alice_engine* e, const alice_buf* b, float* out, size_t len) {
    if (!e || !b || (!out && len)) return fail(ALICE_E_INVALID, "alice_buf_read_f32: null argument");
    if (len > b->len) return fail(ALICE_E_SHAPE, "alice_buf_read_f32: %zu floats from a buffer of %zu", len, b->len);
    CU(cudaMemcpyAsync(out, b->p, len * sizeof(float), cudaMemcpyDeviceToHost, e->stream));
    CU(cudaStreamSynchronize(e->stream));
    return ALICE_OK;
}

int32_t alice_buf_from_device(alice_engine* e, void* dptr, size_t len, alice_buf** out) {
    if (!e || !dptr || !out) return fail(ALICE_E_INVALID, "alice_buf_from_device: null argument");
    if ((uintptr_t)dptr & 15) return fail(ALICE_E_INVALID, "alice_buf_from_device: pointer not 16-byte aligned");
    *out = new alice_buf{e, static_cast<float*>(dptr), len, false};
    alice_engine_retain(e);
    return ALICE_OK;
}

int32_t alice_buf_free(alice_buf* b) {
    if (!b) return ALICE_OK;
    if (b->owned) {
        quiesce(b->e);
        cudaFree(b->p);
    }
    alice_engine_release(b->e);
    delete b;
    return ALICE_OK;
}

}  // extern "C"
