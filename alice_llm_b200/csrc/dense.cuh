// Products with dense bfloat16 weight rows (row-major [rows][cols], cols a multiple of 64, zero-padded by the loader) for
// models whose layers are not in a GGUF block format: one token against two matrices at once (dense_rows.cu), many tokens
// as a tiled product (dense_gemm.cu). Accumulation is in f32 everywhere.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace alice {

using bf16 = __nv_bfloat16;

constexpr uint32_t DENSE_PAD = 64;   // columns of a weight matrix and of the vectors it meets come in multiples of this
inline uint32_t pad_to(uint32_t v, uint32_t m) { return (v + m - 1) / m * m; }

struct DenseMat {
    const bf16* w = nullptr;
    uint32_t n = 0, k = 0;   // rows, (padded) columns
};

enum InputNorm : int { NORM_NONE = 0, NORM_LAYER = 1, NORM_RMS = 2 };

// One token: y0 = W0 h and y1 = act(gate h) * (up h), both of the same h, which every CTA derives from x itself. Either product
// may be absent.
struct RowsIn {
    const float* x = nullptr;
    uint32_t n_x = 0;             // true length; elements [n_x, k) of h are zero
    int norm = NORM_NONE;
    const float* norm_w = nullptr;
    float eps = 0.f;
    DenseMat w0;
    float* y0 = nullptr;
    DenseMat gu;                  // 64 gate rows, 64 up rows, 64 gate rows, ... (gu.n = 2 * ff padded), or empty
    const float *gate_b = nullptr, *up_b = nullptr;   // null: no biases
    float* y1 = nullptr;
    float* h_out = nullptr;       // not x: h itself is left here too, n_x elements
    unsigned long long* argmax_key = nullptr;   // of y0's rows: atomicMax of (order-preserving value, ~row)
};
// One token: out = alpha * x + s1 * (W1 a) + s2 * (W2 f + b2); out and x may be the same vector.
struct RowsOut {
    DenseMat w1, w2;              // w2 may be empty
    float alpha = 1.f;
    const float *a = nullptr, *f = nullptr;
    const float *s1 = nullptr, *s2 = nullptr, *b2 = nullptr;   // s1 null: all ones
    const float* x = nullptr;
    float* out = nullptr;
};
cudaError_t launch_rows_in(const RowsIn& op, int num_sms, cudaStream_t st, bool pdl);
cudaError_t launch_rows_out(const RowsOut& op, int num_sms, cudaStream_t st, bool pdl);

enum DenseEpilogue : int {
    EPI_STORE = 0,     // out[t][n] = acc (and, for n >= col2, a bf16 copy in out2)
    EPI_SWIGLU = 1,    // w holds interleaved gate / up rows; out[t][c] = silu(gate + gate_b) * (up + up_b), biases may be null
    EPI_RESID = 2,     // out[t][n] = alpha * out[t][n] + scale[n] * (acc + bias[n]); scale and bias may be null
    EPI_DECAY = 3,     // out[t][n] = exp(-exp(a_log[n / dim]) * softplus(acc + bias[n]))
    EPI_SIGMOID = 4,   // out[t][n] = sigmoid(acc)
};

// Many tokens: acc[t][n] = sum_k a[t][k] w[n][k], t < tokens.
struct GemmOp {
    uint32_t tokens = 0;
    const void* a = nullptr;      // f32 or bf16 rows, lda elements apart, w.k of them readable
    uint32_t lda = 0;
    bool a_bf16 = false;
    DenseMat w;
    int epi = EPI_STORE;
    void* out = nullptr;
    uint32_t ldo = 0;
    bool out_bf16 = false;
    bf16* out2 = nullptr;
    uint32_t col2 = 0, ld2 = 0;
    const float *bias = nullptr, *bias2 = nullptr, *scale = nullptr, *a_log = nullptr;
    float alpha = 1.f;
    uint32_t dim = 1;
};
// bf16 inputs run on the tensor cores, f32 inputs in f32 arithmetic throughout.
cudaError_t launch_dense_gemm(const GemmOp& op, int num_sms, int* status, cudaStream_t st, bool pdl);

}  // namespace alice
