// Attention of many tokens over a cached latent: keys and values of the whole context have been made from the latent rows,
// the rotated key part is read from the cache itself.
#include "attn_prefill.cuh"

namespace alice {
namespace {

// Queries in bf16 with the rotated part turned to its position. One CTA per token.
__global__ void __launch_bounds__(256) latent_rotate_kernel(const __grid_constant__ LatentArgs a, bf16* out) {
    extern __shared__ float2 cs[];   // (cos, sin) per pair
    const LatentShape& s = a.s;
    const uint32_t t = blockIdx.x, half = s.rot_dims / 2, qd = s.dim + s.rot, n = s.heads * qd;
    pdl_launch_dependents();
    pdl_wait();
    const float p = (float)((uint32_t)*a.pos + t);
    for (uint32_t i = threadIdx.x; i < half; i += 256) {
        float sn, c;
        sincosf(p * a.freq[i], &sn, &c);
        cs[i] = make_float2(c, sn);
    }
    __syncthreads();
    const float* q = a.q + (size_t)t * n;
    for (uint32_t i = threadIdx.x * 2; i < n; i += 512) {   // head sizes are even
        float v[2];
        const uint32_t c = i % qd;
        const float2 x = *reinterpret_cast<const float2*>(q + i);
#pragma unroll
        for (int e = 0; e < 2; e++) {
            v[e] = e ? x.y : x.x;
            if (c + e >= s.dim && c + e < s.dim + s.rot_dims) {
                const uint32_t d = c + e - s.dim;
                if (d < half) v[e] = v[e] * cs[d].x - q[i + e + half] * cs[d].y;
                else v[e] = v[e] * cs[d - half].x + q[i + e - half] * cs[d - half].y;
            }
        }
        *reinterpret_cast<uint32_t*>(out + (size_t)t * n + i) = pack_bf16(v[0], v[1]);
    }
}

}  // namespace

cudaError_t launch_latent_prefill(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (!latent_prefill_fits(a.s) || !a.cache_bf16 || !a.act_bf16) return cudaErrorInvalidValue;
    const cudaError_t err = launch_pdl(latent_rotate_kernel, dim3(tokens), dim3(256), (size_t)(a.s.rot_dims / 2) * sizeof(float2), st, pdl, a, a.q_rot);
    if (err != cudaSuccess) return err;
    const LatentShape& z = a.s;
    PrefillArgs p;
    p.heads = z.heads; p.vdim = p.v_cols = z.vdim; p.q = a.q_rot; p.q_group = z.dim + z.rot; p.q_row = z.heads * p.q_group; p.pos = a.pos; p.sink = a.sink; p.scale = z.scale;
    p.k1 = a.k_all; p.k1_cols = z.dim; p.k1_row = (size_t)z.heads * z.dim; p.k1_head = z.dim;
    p.k2 = static_cast<const bf16*>(a.cache) + z.cp; p.k2_cols = z.rot; p.k2_row = z.cp + z.rp;
    p.v = a.v_all; p.v_row = (size_t)z.heads * z.vdim; p.v_head = z.vdim;
    p.gate = a.y + z.off_g; p.ld_gate = a.ldy; p.out = static_cast<bf16*>(a.out); p.ldo = a.ldo;
    return launch_attn_prefill<false>(p, tokens, st, pdl);
}

}  // namespace alice
