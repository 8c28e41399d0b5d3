// What happens to one accumulated element of a tiled dense product (DenseEpilogue).
#pragma once
#include "dense_dev.cuh"

namespace alice {

template <int EPI>
__device__ __forceinline__ void epi_one(const GemmOp& op, uint32_t t, uint32_t n, float v) {
    const size_t o = (size_t)t * op.ldo + n;
    if constexpr (EPI == EPI_STORE) {
        if (op.out_bf16) put(static_cast<bf16*>(op.out) + o, v);
        else static_cast<float*>(op.out)[o] = v;
        if (op.out2 && n >= op.col2) put(op.out2 + (size_t)t * op.ld2 + (n - op.col2), v);
    } else if constexpr (EPI == EPI_RESID) {
        float* x = static_cast<float*>(op.out) + o;
        const float r = op.bias ? v + op.bias[n] : v;
        *x = op.alpha * *x + (op.scale ? op.scale[n] * r : r);
    } else if constexpr (EPI == EPI_DECAY) {
        static_cast<float*>(op.out)[o] = expf(-expf(op.a_log[n / op.dim]) * softplus_f(v + op.bias[n]));
    } else if constexpr (EPI == EPI_SIGMOID) {
        static_cast<float*>(op.out)[o] = sigmoid_f(v);
    }
}

__device__ __forceinline__ void epi_swiglu(const GemmOp& op, uint32_t t, uint32_t c, float gate, float up) {
    const float v = op.bias ? silu_ref(gate + op.bias[c]) * (up + op.bias2[c]) : silu_ref(gate) * up;
    const size_t o = (size_t)t * op.ldo + c;
    if (op.out_bf16) put(static_cast<bf16*>(op.out) + o, v);
    else static_cast<float*>(op.out)[o] = v;
}

}  // namespace alice
