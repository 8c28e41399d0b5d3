// Device helpers shared by the dense-weight kernels and the layer kernels built on them.
#pragma once
#include "common.cuh"
#include "dense.cuh"

namespace alice {

__device__ __forceinline__ float sigmoid_f(float z) { return __fdiv_rn(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
// tanh(x / (2 log2(e))), from the exponential: exact to an ulp or two of 1
__device__ __forceinline__ float tanh_of_pow2(float x) { return 1.0f - __fdividef(2.0f, 1.0f + exp2f(x)); }
__device__ __forceinline__ float2 bf2(uint32_t u) { return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u)); }
__device__ __forceinline__ float dot8(uint4 v, float4 x0, float4 x1, float acc) {
    const float2 a = bf2(v.x), b = bf2(v.y), d = bf2(v.z), e = bf2(v.w);
    acc = fmaf(a.x, x0.x, acc); acc = fmaf(a.y, x0.y, acc); acc = fmaf(b.x, x0.z, acc); acc = fmaf(b.y, x0.w, acc);
    acc = fmaf(d.x, x1.x, acc); acc = fmaf(d.y, x1.y, acc); acc = fmaf(e.x, x1.z, acc); acc = fmaf(e.y, x1.w, acc);
    return acc;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float get(const float* p) { return *p; }
__device__ __forceinline__ float get(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// Sum over the block (NW warps), the same value in every thread; `red` holds NW floats.
template <int NW>
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.0f;
#pragma unroll
    for (int i = 0; i < NW; i++) s += red[i];
    __syncthreads();
    return s;
}

// h[0 .. k) (shared memory) <- norm(x[0 .. n)) * w, zero beyond n.
template <int NW>
__device__ __forceinline__ void load_normed(float* h, const float* x, uint32_t n, uint32_t k, int norm, const float* w, float eps, float* red) {
    float s = 0.0f;
    for (uint32_t i = threadIdx.x; i < k; i += NW * 32) {
        const float v = i < n ? __ldcg(x + i) : 0.0f;
        h[i] = v;
        s += norm == NORM_LAYER ? v : v * v;
    }
    if (norm == NORM_NONE) { __syncthreads(); return; }
    s = block_sum<NW>(s, red);
    float mean = 0.0f;
    if (norm == NORM_LAYER) {
        mean = s / (float)n;
        float q = 0.0f;
        for (uint32_t i = threadIdx.x; i < n; i += NW * 32) { const float d = h[i] - mean; q += d * d; }
        s = block_sum<NW>(q, red);
    }
    const float inv = __frcp_rn(__fsqrt_rn(s / (float)n + eps));
    for (uint32_t i = threadIdx.x; i < n; i += NW * 32) h[i] = (h[i] - mean) * inv * w[i];
    __syncthreads();
}

inline void pdl_config(cudaLaunchConfig_t& lc, cudaLaunchAttribute* at, dim3 grid, dim3 block, size_t smem, cudaStream_t st, bool pdl) {
    lc = {};
    lc.gridDim = grid; lc.blockDim = block; lc.dynamicSmemBytes = smem; lc.stream = st;
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = 1;
    lc.attrs = at; lc.numAttrs = pdl ? 1 : 0;
}
template <class K, class... A>
cudaError_t launch_pdl(K kern, dim3 grid, dim3 block, size_t smem, cudaStream_t st, bool pdl, A... args) {
    cudaLaunchConfig_t lc; cudaLaunchAttribute at[1];
    pdl_config(lc, at, grid, block, smem, st, pdl);
    return cudaLaunchKernelEx(&lc, kern, args...);
}
// Raises a kernel's dynamic shared memory limit once per device.
template <class K>
cudaError_t allow_smem(K kern, size_t bytes, bool (&done)[64]) {
    int dev = 0;
    cudaError_t err = cudaGetDevice(&dev);
    if (err != cudaSuccess) return err;
    if (dev >= 0 && dev < 64 && done[dev]) return cudaSuccess;
    err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (err == cudaSuccess && dev >= 0 && dev < 64) done[dev] = true;
    return err;
}

}  // namespace alice
