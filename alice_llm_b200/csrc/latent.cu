// Attention over a cached latent: one row [latent c | rotated key part] per token serves every head. Queries are taken into
// the latent space (W_uk^T q), so scores and weighted sums run on the cached rows themselves and the values are made once
// per query from the weighted latent (W_uv c). A learned number per head joins the softmax denominator.
#include "dense_dev.cuh"
#include "mixers.cuh"

namespace alice {
namespace {

__device__ __forceinline__ void rotate_pair(float u, float v, float angle, float& a, float& b) {
    float s, c;
    sincosf(angle, &s, &c);
    a = u * c - v * s;
    b = v * c + u * s;
}

// Norm of the key latent and the rotated key part into the cache (a block of NT threads).
template <class CT, int NT>
__device__ __forceinline__ void cache_append(const LatentArgs& a, uint32_t t, float* red) {
    const LatentShape& s = a.s;
    const uint32_t p = (uint32_t)*a.pos + t;
    const float* y = a.y + (size_t)t * a.ldy + s.off_kv;
    float q = 0.0f;
    for (uint32_t i = threadIdx.x; i < s.kv_rank; i += NT) q = fmaf(y[i], y[i], q);
    q = block_sum<NT / 32>(q, red);
    const float inv = __frcp_rn(__fsqrt_rn(q / (float)s.kv_rank + a.eps));
    CT* row = static_cast<CT*>(a.cache) + (size_t)p * (s.cp + s.rp);
    for (uint32_t i = threadIdx.x; i < s.kv_rank; i += NT) put(row + i, y[i] * inv * a.kv_norm[i]);
    const float* kr = y + s.kv_rank;
    const uint32_t half = s.rot_dims / 2;
    for (uint32_t i = threadIdx.x; i < half; i += NT) {
        float u, v;
        rotate_pair(kr[i], kr[half + i], (float)p * a.freq[i], u, v);
        put(row + s.cp + i, u);
        put(row + s.cp + half + i, v);
    }
    for (uint32_t i = s.rot_dims + threadIdx.x; i < s.rot; i += NT) put(row + s.cp + i, kr[i]);
}

// One CTA per token: norm of the query latent, and the token's cache row.
template <class OT, class CT>
__global__ void __launch_bounds__(128) latent_norm_kernel(const __grid_constant__ LatentArgs a) {
    __shared__ float red[4];
    pdl_launch_dependents();
    pdl_wait();
    const LatentShape& s = a.s;
    const uint32_t t = blockIdx.x;
    const float* y = a.y + (size_t)t * a.ldy + s.off_q;
    float q = 0.0f;
    for (uint32_t i = threadIdx.x; i < s.q_rank; i += 128) q = fmaf(y[i], y[i], q);
    q = block_sum<4>(q, red);
    const float inv = __frcp_rn(__fsqrt_rn(q / (float)s.q_rank + a.eps));
    OT* cq = static_cast<OT*>(a.cqn) + (size_t)t * s.qp;
    for (uint32_t i = threadIdx.x; i < s.qp; i += 128) put(cq + i, i < s.q_rank ? y[i] * inv * a.q_norm[i] : 0.0f);
    cache_append<CT, 128>(a, t, red);
}

// grid (heads, cp / 64, tokens): 64 latent columns of one head's query; the first slice also rotates the rotated part. With
// a.append one more row of CTAs (blockIdx.x == heads, first slice) makes the token's cache row.
template <class CT>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const __grid_constant__ LatentArgs a) {
    extern __shared__ __align__(16) float sm[];   // query [dim], then 4 x 64 partial sums
    const LatentShape& s = a.s;
    const uint32_t h = blockIdx.x, c0 = blockIdx.y * 64, t = blockIdx.z;
    float* qs = sm;
    float* part = sm + ((s.dim + 3) & ~3u);
    pdl_launch_dependents();
    if (h == s.heads) {
        pdl_wait();
        if (blockIdx.y == 0) cache_append<CT, 256>(a, t, part);
        return;
    }
    const bf16* w = a.uk + (size_t)h * s.dim * s.cp + c0;
    // a thread sums 8 columns over every 32nd row; rows of the first round travel ahead of the wait
    const uint32_t cg = threadIdx.x & 7, dr = threadIdx.x >> 3;
    for (uint32_t d = dr; d < s.dim; d += 32) prefetch_l2(w + (size_t)d * s.cp + cg * 8);
    pdl_wait();
    const float* q = a.q + ((size_t)t * s.heads + h) * (s.dim + s.rot);
    float* out = a.ql + ((size_t)t * s.heads + h) * (s.cp + s.rp);
    for (uint32_t i = threadIdx.x; i < s.dim; i += 256) qs[i] = q[i];
    __syncthreads();
    float acc[8] = {};
#pragma unroll 4
    for (uint32_t d = dr; d < s.dim; d += 32) {
        const uint4 v = __ldg(reinterpret_cast<const uint4*>(w + (size_t)d * s.cp + cg * 8));
        const float x = qs[d];
        const float2 e0 = bf2(v.x), e1 = bf2(v.y), e2 = bf2(v.z), e3 = bf2(v.w);
        acc[0] = fmaf(e0.x, x, acc[0]); acc[1] = fmaf(e0.y, x, acc[1]); acc[2] = fmaf(e1.x, x, acc[2]); acc[3] = fmaf(e1.y, x, acc[3]);
        acc[4] = fmaf(e2.x, x, acc[4]); acc[5] = fmaf(e2.y, x, acc[5]); acc[6] = fmaf(e3.x, x, acc[6]); acc[7] = fmaf(e3.y, x, acc[7]);
    }
    // lanes 8 apart in a warp share columns
#pragma unroll
    for (int i = 0; i < 8; i++) {
        acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 8);
        acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 16);
    }
    const uint32_t warp = threadIdx.x >> 5;
    if ((threadIdx.x & 31) < 8)
#pragma unroll
        for (int i = 0; i < 8; i++) part[warp * 64 + cg * 8 + i] = acc[i];
    __syncthreads();
    if (threadIdx.x < 64) {
        float v = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; i++) v += part[i * 64 + threadIdx.x];
        out[c0 + threadIdx.x] = v;
    }
    if (blockIdx.y == 0) {
        const float p = (float)((uint32_t)*a.pos + t);
        const uint32_t half = s.rot_dims / 2;
        const float* r = q + s.dim;
        for (uint32_t i = threadIdx.x; i < s.rp; i += 256) {
            float v = 0.0f;
            if (i < s.rot_dims) {
                float b0, b1;
                const uint32_t j = i < half ? i : i - half;
                rotate_pair(r[j], r[half + j], p * a.freq[j], b0, b1);
                v = i < half ? b0 : b1;
            } else if (i < s.rot) {
                v = r[i];
            }
            out[s.cp + i] = v;
        }
    }
}

// f32 attention of latent-space queries over the cached rows. grid (head groups, splits, tokens), 8 warps; a warp owns RW
// heads, a lane one of the 32 keys of a tile (scores) and NC latent columns 32 apart (weighted sum).
constexpr int ATT_KEYS = 32;
template <class CT, int RW, int NC>
__global__ void __launch_bounds__(256) latent_attn_kernel(const __grid_constant__ LatentArgs a) {
    extern __shared__ __align__(16) float sm[];
    const LatentShape& s = a.s;
    const uint32_t width = s.cp + s.rp, ldk = width + 4, rows = 8 * RW;
    float* qs = sm;                       // [rows][width]
    float* ks = sm + (size_t)rows * width;   // [32][width + 4]
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.z, h0 = blockIdx.x * rows;
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t ctx = (uint32_t)*a.pos + t + 1;
    const uint32_t share = ((ctx + gridDim.y - 1) / gridDim.y + ATT_KEYS - 1) / ATT_KEYS * ATT_KEYS;
    const uint32_t lo = min(ctx, blockIdx.y * share), hi = min(ctx, lo + share);
    for (uint32_t i = threadIdx.x; i < rows * width; i += 256) {
        const uint32_t h = h0 + i / width;
        qs[i] = h < s.heads ? a.ql[((size_t)t * s.heads + h) * width + i % width] * s.scale : 0.0f;
    }
    float m[RW], l[RW], o[RW][NC];
#pragma unroll
    for (int r = 0; r < RW; r++) {
        m[r] = -INFINITY; l[r] = 0.0f;
#pragma unroll
        for (int i = 0; i < NC; i++) o[r][i] = 0.0f;
    }
    const CT* cache = static_cast<const CT*>(a.cache);
    for (uint32_t k0 = lo; k0 < hi; k0 += ATT_KEYS) {
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < ATT_KEYS * (width / 4); i += 256) {
            const uint32_t j = i / (width / 4), d = i % (width / 4) * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (k0 + j < hi) {
                const CT* src = cache + (size_t)(k0 + j) * width + d;
                if constexpr (sizeof(CT) == 4) {
                    v = *reinterpret_cast<const float4*>(src);
                } else {
                    const uint2 u = *reinterpret_cast<const uint2*>(src);
                    const float2 x = bf2(u.x), y = bf2(u.y);
                    v = make_float4(x.x, x.y, y.x, y.y);
                }
            }
            *reinterpret_cast<float4*>(ks + (size_t)j * ldk + d) = v;
        }
        __syncthreads();
        float sc[RW];
#pragma unroll
        for (int r = 0; r < RW; r++) sc[r] = 0.0f;
        const float* kp = ks + (size_t)lane * ldk;
        const float* qp = qs + (size_t)warp * RW * width;
        for (uint32_t d = 0; d < width; d += 4) {
            const float4 k = *reinterpret_cast<const float4*>(kp + d);
#pragma unroll
            for (int r = 0; r < RW; r++) {
                const float4 q = *reinterpret_cast<const float4*>(qp + (size_t)r * width + d);
                sc[r] = fmaf(q.x, k.x, sc[r]); sc[r] = fmaf(q.y, k.y, sc[r]); sc[r] = fmaf(q.z, k.z, sc[r]); sc[r] = fmaf(q.w, k.w, sc[r]);
            }
        }
        float p[RW];
#pragma unroll
        for (int r = 0; r < RW; r++) {
            const float v = k0 + lane < hi ? sc[r] : -INFINITY;
            const float top = fmaxf(m[r], warp_max(v)), f = expf(m[r] - top);   // a tile holds at least one key
            p[r] = expf(v - top);
            l[r] = fmaf(l[r], f, warp_sum(p[r]));
            m[r] = top;
#pragma unroll
            for (int i = 0; i < NC; i++) o[r][i] *= f;
        }
        for (uint32_t j = 0; j < ATT_KEYS; j++) {
            float pj[RW];
#pragma unroll
            for (int r = 0; r < RW; r++) pj[r] = __shfl_sync(0xffffffffu, p[r], j);
            const float* c = ks + (size_t)j * ldk + lane;
#pragma unroll
            for (int i = 0; i < NC; i++) {
                const float v = 32 * i + lane < s.cp ? c[32 * i] : 0.0f;
#pragma unroll
                for (int r = 0; r < RW; r++) o[r][i] = fmaf(pj[r], v, o[r][i]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < RW; r++) {
        const uint32_t h = h0 + warp * RW + r;
        if (h >= s.heads) break;
        float* out = a.part + (((size_t)t * gridDim.y + blockIdx.y) * s.heads + h) * (s.cp + 2);
#pragma unroll
        for (int i = 0; i < NC; i++)
            if (32 * i + lane < s.cp) out[32 * i + lane] = o[r][i];
        if (lane == 0) { out[s.cp] = m[r]; out[s.cp + 1] = l[r]; }
    }
}

// Joins the shares of the context and the sink: weighted latent of every head. grid (heads, cp / 64, tokens), 256 threads: 64
// columns, the shares dealt to four groups.
__global__ void __launch_bounds__(256) latent_join_kernel(const __grid_constant__ LatentArgs a) {
    extern __shared__ float wt[];   // one weight per share
    __shared__ float sum[4][64];
    const LatentShape& s = a.s;
    const uint32_t h = blockIdx.x, t = blockIdx.z, lane = threadIdx.x & 31, g = threadIdx.x >> 6, c = blockIdx.y * 64 + (threadIdx.x & 63);
    pdl_launch_dependents();
    pdl_wait();
    const float* part = a.part + ((size_t)t * a.splits * s.heads + h) * (s.cp + 2);
    const size_t step = (size_t)s.heads * (s.cp + 2);
    // shares that can hold keys (both attention kernels hand out the context in whole tiles of at least 32)
    const uint32_t ctx = (uint32_t)*a.pos + t + 1, shares = min(a.splits, (ctx + 31) / 32);
    if (threadIdx.x < 32) {
        float top = a.sink[h];
        for (uint32_t i = lane; i < shares; i += 32) top = fmaxf(top, part[i * step + s.cp]);
        top = warp_max(top);
        float den = 0.0f;
        for (uint32_t i = lane; i < shares; i += 32) {
            const float f = expf(part[i * step + s.cp] - top);   // an empty share left -inf
            wt[i] = f;
            den = fmaf(f, part[i * step + s.cp + 1], den);
        }
        den = warp_sum(den) + expf(a.sink[h] - top);
        const float inv = __frcp_rn(den);
        for (uint32_t i = lane; i < shares; i += 32) wt[i] *= inv;
    }
    __syncthreads();
    float v = 0.0f;
#pragma unroll 16
    for (uint32_t k = g; k < shares; k += 4) {
        const float x = part[k * step + c], w = wt[k];
        v = w != 0.0f ? fmaf(w, x, v) : v;   // an empty share holds no sums
    }
    sum[g][threadIdx.x & 63] = v;
    __syncthreads();
    if (g == 0) a.mix[((size_t)t * s.heads + h) * s.cp + c] = (sum[0][threadIdx.x] + sum[1][threadIdx.x]) + (sum[2][threadIdx.x] + sum[3][threadIdx.x]);
}

// Value rows of the weighted latent and the output gate. grid (heads, groups of 16 rows, tokens), 8 warps of two rows.
template <class OT>
__global__ void __launch_bounds__(256) latent_value_kernel(const __grid_constant__ LatentArgs a) {
    extern __shared__ __align__(16) float c[];   // latent [cp]
    const LatentShape& s = a.s;
    const uint32_t h = blockIdx.x, t = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, r0 = blockIdx.y * 16 + warp;
    const bf16* uv = a.uv + (size_t)h * s.vdim * s.cp;
    pdl_launch_dependents();
    for (uint32_t r = r0; r < min(s.vdim, r0 + 16); r += 8)
        for (uint32_t i = lane * 64; i < s.cp; i += 32 * 64) prefetch_l2(uv + (size_t)r * s.cp + i);
    pdl_wait();
    const float* mix = a.mix + ((size_t)t * s.heads + h) * s.cp;
    for (uint32_t i = threadIdx.x; i < s.cp; i += 256) c[i] = mix[i];
    __syncthreads();
    const float* gate = a.y + (size_t)t * a.ldy + s.off_g + (size_t)h * s.vdim;
    OT* out = static_cast<OT*>(a.out) + (size_t)t * a.ldo + (size_t)h * s.vdim;
    for (uint32_t r = r0; r < min(s.vdim, r0 + 16); r += 8) {
        float v = 0.0f;
        for (uint32_t i = lane * 8; i < s.cp; i += 256) {
            const uint4 w = __ldg(reinterpret_cast<const uint4*>(uv + (size_t)r * s.cp + i));
            const float2 e0 = bf2(w.x), e1 = bf2(w.y), e2 = bf2(w.z), e3 = bf2(w.w);
            v = fmaf(e0.x, c[i], v); v = fmaf(e0.y, c[i + 1], v); v = fmaf(e1.x, c[i + 2], v); v = fmaf(e1.y, c[i + 3], v);
            v = fmaf(e2.x, c[i + 4], v); v = fmaf(e2.y, c[i + 5], v); v = fmaf(e3.x, c[i + 6], v); v = fmaf(e3.y, c[i + 7], v);
        }
        v = warp_sum(v);
        if (lane == 0) put(out + r, v * sigmoid_f(gate[r]));
    }
    if (h + 1 == s.heads && blockIdx.y == 0)   // padding up to the stride
        for (uint32_t i = s.vdim + threadIdx.x; i < a.ldo - h * s.vdim; i += 256) put(out + i, 0.0f);
}

template <class CT, int RW, int NC>
cudaError_t attn_inst(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    const cudaError_t err = allow_smem(latent_attn_kernel<CT, RW, NC>, 224 * 1024, done);
    if (err != cudaSuccess) return err;
    const uint32_t width = a.s.cp + a.s.rp;
    const size_t smem = ((size_t)8 * RW * width + (size_t)ATT_KEYS * (width + 4)) * 4;
    if (smem > 224 * 1024) return cudaErrorInvalidValue;
    return launch_pdl(latent_attn_kernel<CT, RW, NC>, dim3((a.s.heads + 8 * RW - 1) / (8 * RW), a.splits, tokens), dim3(256), smem, st, pdl, a);
}
template <class CT>
cudaError_t attn_type(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const bool few = a.s.heads <= 8;
    if (a.s.cp <= 128) return few ? attn_inst<CT, 1, 4>(a, tokens, st, pdl) : attn_inst<CT, 4, 4>(a, tokens, st, pdl);
    if (a.s.cp <= 512) return few ? attn_inst<CT, 1, 16>(a, tokens, st, pdl) : attn_inst<CT, 4, 16>(a, tokens, st, pdl);
    if (a.s.cp <= 1024) return attn_inst<CT, 1, 32>(a, tokens, st, pdl);
    return cudaErrorInvalidValue;
}

}  // namespace

cudaError_t launch_latent_norm(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (a.act_bf16) return launch_pdl(latent_norm_kernel<bf16, bf16>, dim3(tokens), dim3(128), 0, st, pdl, a);
    return a.cache_bf16 ? launch_pdl(latent_norm_kernel<float, bf16>, dim3(tokens), dim3(128), 0, st, pdl, a)
                        : launch_pdl(latent_norm_kernel<float, float>, dim3(tokens), dim3(128), 0, st, pdl, a);
}
cudaError_t launch_latent_absorb(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const dim3 grid(a.s.heads + (a.append ? 1 : 0), a.s.cp / 64, tokens);
    const size_t smem = (size_t)(((a.s.dim + 3) & ~3u) + 512) * 4;
    return a.cache_bf16 ? launch_pdl(latent_absorb_kernel<bf16>, grid, dim3(256), smem, st, pdl, a)
                        : launch_pdl(latent_absorb_kernel<float>, grid, dim3(256), smem, st, pdl, a);
}
cudaError_t launch_latent_attn(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (a.cache_bf16 && latent_decode_fits(a.s)) return launch_latent_decode(a, tokens, st, pdl);
    return a.cache_bf16 ? attn_type<bf16>(a, tokens, st, pdl) : attn_type<float>(a, tokens, st, pdl);
}
cudaError_t launch_latent_out(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const cudaError_t err = launch_pdl(latent_join_kernel, dim3(a.s.heads, a.s.cp / 64, tokens), dim3(256), (size_t)a.splits * 4, st, pdl, a);
    if (err != cudaSuccess) return err;
    const dim3 grid(a.s.heads, (a.s.vdim + 15) / 16, tokens);
    return a.act_bf16 ? launch_pdl(latent_value_kernel<bf16>, grid, dim3(256), (size_t)a.s.cp * 4, st, pdl, a)
                      : launch_pdl(latent_value_kernel<float>, grid, dim3(256), (size_t)a.s.cp * 4, st, pdl, a);
}

}  // namespace alice
