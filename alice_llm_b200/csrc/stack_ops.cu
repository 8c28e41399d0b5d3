// Small per-token kernels of layer-stack models: the embedding (and what re-enters the stream before a looped pass) and the
// layer norm ahead of a tiled product.
#include "dense_dev.cuh"
#include "mixers.cuh"

namespace alice {
namespace {

__global__ void __launch_bounds__(1024) enter_kernel(const __grid_constant__ EnterArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t t = blockIdx.x;
    uint32_t tok = a.emb ? (uint32_t)a.tokens[t] : 0u;
    if (tok >= a.vocab) tok = 0;
    const bf16* e = a.emb ? a.emb + (size_t)tok * a.emb_ld : nullptr;
    float* x = a.x + (size_t)t * a.ld;
    for (uint32_t i = threadIdx.x; i < a.n; i += blockDim.x) {
        float v = a.set ? 0.0f : x[i];
        if (e) v += __fmul_rn(__bfloat162float(e[i]), a.scale);
        if (a.step) v += a.step[i];
        x[i] = v;
    }
}

template <class OT>
__global__ void __launch_bounds__(256) layer_norm_kernel(const __grid_constant__ NormArgs a) {
    extern __shared__ __align__(16) float h[];
    __shared__ float red[8];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t t = blockIdx.x, src = a.gather ? a.idx[t] : t;
    load_normed<8>(h, a.x + (size_t)src * a.ldx, a.n, a.k, NORM_LAYER, a.w, a.eps, red);
    OT* out = static_cast<OT*>(a.out) + (size_t)t * a.k;
    for (uint32_t i = threadIdx.x; i < a.k; i += 256) put(out + i, h[i]);
}

}  // namespace

cudaError_t launch_enter(const EnterArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    return launch_pdl(enter_kernel, dim3(tokens), dim3(a.n > 512 ? 1024 : 256), 0, st, pdl, a);
}

cudaError_t launch_layer_norm(const NormArgs& a, uint32_t rows, cudaStream_t st, bool pdl) {
    if (a.gather && rows > MAX_NORM_ROWS) return cudaErrorInvalidValue;
    static bool done_f[64] = {}, done_b[64] = {};
    cudaError_t err = a.out_bf16 ? allow_smem(layer_norm_kernel<bf16>, 224 * 1024, done_b) : allow_smem(layer_norm_kernel<float>, 224 * 1024, done_f);
    if (err != cudaSuccess) return err;
    return a.out_bf16 ? launch_pdl(layer_norm_kernel<bf16>, dim3(rows), dim3(256), (size_t)a.k * 4, st, pdl, a)
                      : launch_pdl(layer_norm_kernel<float>, dim3(rows), dim3(256), (size_t)a.k * 4, st, pdl, a);
}

}  // namespace alice
