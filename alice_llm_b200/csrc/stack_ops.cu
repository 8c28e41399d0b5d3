// Small per-token kernels of layer-stack models: the embedding (and what re-enters the stream before a looped pass) and the
// norms ahead of or behind a tiled product.
#include "dense_dev.cuh"
#include "mixers.cuh"
#include "mma_sync.cuh"

namespace alice {
namespace {

__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(bf16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w)); }

template <class HT>
__global__ void __launch_bounds__(256) enter_kernel(const __grid_constant__ EnterArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t t = blockIdx.x;
    uint32_t tok = a.emb ? (uint32_t)a.tokens[t] : 0u;
    if (tok >= a.vocab) tok = 0;
    const bf16* e = a.emb ? a.emb + (size_t)tok * a.emb_ld : nullptr;
    float* x = a.x + (size_t)t * a.ld;
    for (uint32_t c = threadIdx.x * 4; c < a.ld; c += 1024) {   // rows are padded with zeros to a multiple of 64
        float4 v = a.set ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(x + c);
        if (e) {
            const uint2 u = __ldg(reinterpret_cast<const uint2*>(e + c));
            const float2 p = bf2(u.x), q = bf2(u.y);
            v.x += __fmul_rn(p.x, a.scale); v.y += __fmul_rn(p.y, a.scale); v.z += __fmul_rn(q.x, a.scale); v.w += __fmul_rn(q.y, a.scale);
        }
        if (a.step) {
            if (c < a.n) v.x += a.step[c];
            if (c + 1 < a.n) v.y += a.step[c + 1];
            if (c + 2 < a.n) v.z += a.step[c + 2];
            if (c + 3 < a.n) v.w += a.step[c + 3];
        }
        *reinterpret_cast<float4*>(x + c) = v;
        if (a.h) put4(static_cast<HT*>(a.h) + (size_t)t * a.ld + c, v);
    }
}

// The row is held in registers: a thread owns every 256th group of four elements (NV groups; rows up to 1024 * NV wide).
template <class OT, int NV>
__global__ void __launch_bounds__(256) norm_kernel(const __grid_constant__ NormArgs a) {
    __shared__ float red[8];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t t = blockIdx.x, src = a.gather ? a.idx[t] : t;
    const float* x = a.x + (size_t)src * a.ldx;
    float v[NV][4];
    float s = 0.0f;
#pragma unroll
    for (int j = 0; j < NV; j++) {
        const uint32_t c = (threadIdx.x + j * 256) * 4;
        const float4 u = c < a.k ? *reinterpret_cast<const float4*>(x + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[j][0] = u.x; v[j][1] = u.y; v[j][2] = u.z; v[j][3] = u.w;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            if (c + i >= a.n) v[j][i] = 0.0f;
            s += a.norm == NORM_LAYER ? v[j][i] : v[j][i] * v[j][i];
        }
    }
    float mean = 0.0f, inv = 1.0f;
    if (a.norm != NORM_NONE) {
        s = block_sum<8>(s, red);
        if (a.norm == NORM_LAYER) {
            mean = s / (float)a.n;
            float q = 0.0f;
#pragma unroll
            for (int j = 0; j < NV; j++)
#pragma unroll
                for (int i = 0; i < 4; i++)
                    if ((threadIdx.x + j * 256) * 4 + i < a.n) { const float d = v[j][i] - mean; q += d * d; }
            s = block_sum<8>(q, red);
        }
        inv = __frcp_rn(__fsqrt_rn(s / (float)a.n + a.eps));
    }
    OT* out = static_cast<OT*>(a.out) + (size_t)t * a.k;
#pragma unroll
    for (int j = 0; j < NV; j++) {
        const uint32_t c = (threadIdx.x + j * 256) * 4;
        if (c >= a.k) break;
        if (a.norm != NORM_NONE)
#pragma unroll
            for (int i = 0; i < 4; i++) v[j][i] = c + i < a.n ? (v[j][i] - mean) * inv * a.w[c + i] : 0.0f;
        const float4 u = make_float4(v[j][0], v[j][1], v[j][2], v[j][3]);
        if (a.out) put4(out + c, u);
        if (a.x_out) put4(a.x_out + (size_t)t * a.ldx + c, u);
    }
}

template <class OT>
cudaError_t norm_type(const NormArgs& a, uint32_t rows, cudaStream_t st, bool pdl) {
    if (a.k <= 1024) return launch_pdl(norm_kernel<OT, 1>, dim3(rows), dim3(256), 0, st, pdl, a);
    if (a.k <= 4096) return launch_pdl(norm_kernel<OT, 4>, dim3(rows), dim3(256), 0, st, pdl, a);
    if (a.k <= 16384) return launch_pdl(norm_kernel<OT, 16>, dim3(rows), dim3(256), 0, st, pdl, a);
    return launch_pdl(norm_kernel<OT, 56>, dim3(rows), dim3(256), 0, st, pdl, a);
}

}  // namespace

cudaError_t launch_enter(const EnterArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (a.ld % 4 || a.ld < a.n || (a.emb && a.emb_ld < a.ld)) return cudaErrorInvalidValue;
    return a.h_bf16 ? launch_pdl(enter_kernel<bf16>, dim3(tokens), dim3(256), 0, st, pdl, a) : launch_pdl(enter_kernel<float>, dim3(tokens), dim3(256), 0, st, pdl, a);
}

cudaError_t launch_norm(const NormArgs& a, uint32_t rows, cudaStream_t st, bool pdl) {
    if ((a.gather && rows > MAX_NORM_ROWS) || a.k % 4 || a.ldx % 4 || a.k > 56 * 1024 || a.ldx < a.k || (a.gather && a.x_out)) return cudaErrorInvalidValue;
    return a.out_bf16 ? norm_type<bf16>(a, rows, st, pdl) : norm_type<float>(a, rows, st, pdl);
}

}  // namespace alice
