// Attention whose key / value heads serve groups of query heads (a plain key / value cache): rotation and norm of queries and
// keys into place, and the f32 form for any number of tokens.
#include "grouped_dev.cuh"

namespace alice {
namespace {

// One CTA per token; a warp per row of a head: queries, then keys, then values. The next row is loaded while one is finished.
template <class CT, int E>
__global__ void __launch_bounds__(256) grouped_prepare_kernel(const __grid_constant__ GroupedArgs a) {
    __shared__ float2 cs[GROUPED_PAIRS];
    const GroupedShape& s = a.s;
    const uint32_t t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, group = s.heads / s.kv_heads, rows = s.heads + 2 * s.kv_heads;
    pdl_launch_dependents();
    pdl_wait();
    const float* y = a.y + (size_t)t * a.ldy;
    HeadRow<E> row[2];
    auto load = [&](uint32_t i, HeadRow<E>& r) {
        if (i < s.heads) r.load(y + (size_t)i * s.dim, s.dim, s.rot_dims, lane);
        else if (i < s.heads + s.kv_heads) r.load(y + s.off_k + (size_t)(i - s.heads) * s.dim, s.dim, s.rot_dims, lane);
        else if (i < rows) r.load(y + s.off_v + (size_t)(i - s.heads - s.kv_heads) * s.vdim, s.vdim, 0, lane);
    };
    load(warp, row[0]);
    const uint32_t p = (uint32_t)*a.pos + t;
    rotation_table(cs, a.freq, s.rot_dims / 2, p, 256);
    __syncthreads();
    auto store = [&](uint32_t i, HeadRow<E>& r) {
        if (i < s.heads) {
            r.store(static_cast<CT*>(a.q) + ((size_t)(i / group * gridDim.x + t) * group + i % group) * s.dp, s.dp, s.unit_qk, cs, a.eps, lane);
        } else {
            const bool key = i < s.heads + s.kv_heads;
            CT* out = static_cast<CT*>(a.cache) + ((size_t)(i - s.heads - (key ? 0 : s.kv_heads)) * a.plane_rows + p) * s.ld();
            r.store(key ? out : out + s.dp, key ? s.dp : s.vp, key && s.unit_qk, cs, a.eps, lane);
        }
    };
    for (uint32_t i = warp; i < rows; i += 16) {
        load(i + 8, row[1]);
        store(i, row[0]);
        load(i + 16, row[0]);
        if (i + 8 < rows) store(i + 8, row[1]);
    }
}
template <class CT>
cudaError_t prepare_type(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const uint32_t n = std::max(a.s.dp, a.s.vp);
    if (n <= 64) return launch_pdl(grouped_prepare_kernel<CT, 2>, dim3(tokens), dim3(256), 0, st, pdl, a);
    if (n <= 128) return launch_pdl(grouped_prepare_kernel<CT, 4>, dim3(tokens), dim3(256), 0, st, pdl, a);
    if (n <= 256) return launch_pdl(grouped_prepare_kernel<CT, 8>, dim3(tokens), dim3(256), 0, st, pdl, a);
    return launch_pdl(grouped_prepare_kernel<CT, 16>, dim3(tokens), dim3(256), 0, st, pdl, a);
}

// f32 arithmetic. grid (blocks of rows, kv_heads), 8 warps of RW rows; a row is one (token, head of the group), a lane one of the
// 32 keys of a tile (scores) and NC value columns 32 apart (weighted sum). The sink is the state the online softmax starts from.
constexpr uint32_t GA_KEYS = 32, GA_RW = 4, GA_ROWS = 8 * GA_RW;
template <class CT, class OT, int NC>
__global__ void __launch_bounds__(256) grouped_attn_kernel(const __grid_constant__ GroupedArgs a, uint32_t tokens) {
    extern __shared__ __align__(16) float sm[];
    const GroupedShape& s = a.s;
    const uint32_t width = s.dp + s.vp, ldk = width + 4, ldc = s.ld(), group = s.heads / s.kv_heads;
    float* qs = sm;                                  // [GA_ROWS][dp]
    float* ks = sm + (size_t)GA_ROWS * s.dp;         // [GA_KEYS][width + 4]
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, kh = blockIdx.y, r0 = blockIdx.x * GA_ROWS, rows = tokens * group;
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t p0 = (uint32_t)*a.pos, last = min(r0 + GA_ROWS, rows) - 1, keys = p0 + last / group + 1;
    for (uint32_t i = threadIdx.x; i < GA_ROWS * s.dp; i += 256) {
        const uint32_t r = r0 + i / s.dp;
        qs[i] = r < rows ? get(static_cast<const CT*>(a.q) + ((size_t)kh * rows + r) * s.dp + i % s.dp) * s.scale : 0.0f;
    }
    float m[GA_RW], l[GA_RW], o[GA_RW][NC];
    uint32_t see[GA_RW];                             // keys the row sees
#pragma unroll
    for (int r = 0; r < (int)GA_RW; r++) {
        const uint32_t row = min(r0 + warp * GA_RW + r, last);
        m[r] = a.sink[kh * group + row % group]; l[r] = 1.0f; see[r] = p0 + row / group + 1;
#pragma unroll
        for (int i = 0; i < NC; i++) o[r][i] = 0.0f;
    }
    const CT* plane = static_cast<const CT*>(a.cache) + (size_t)kh * a.plane_rows * ldc;
    for (uint32_t k0 = 0; k0 < keys; k0 += GA_KEYS) {
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < GA_KEYS * (width / 4); i += 256) {
            const uint32_t j = i / (width / 4), d = i % (width / 4) * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (k0 + j < keys) {
                const CT* src = plane + (size_t)(k0 + j) * ldc + d;
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
        float p[GA_RW] = {};
        const float* kp = ks + (size_t)lane * ldk;
        const float* qp = qs + (size_t)warp * GA_RW * s.dp;
        for (uint32_t d = 0; d < s.dp; d += 4) {
            const float4 k = *reinterpret_cast<const float4*>(kp + d);
#pragma unroll
            for (int r = 0; r < (int)GA_RW; r++) {
                const float4 q = *reinterpret_cast<const float4*>(qp + (size_t)r * s.dp + d);
                p[r] = fmaf(q.x, k.x, p[r]); p[r] = fmaf(q.y, k.y, p[r]); p[r] = fmaf(q.z, k.z, p[r]); p[r] = fmaf(q.w, k.w, p[r]);
            }
        }
#pragma unroll
        for (int r = 0; r < (int)GA_RW; r++) {
            float v = p[r];
            if (s.softcap > 0.0f) v = s.softcap * tanhf(v / s.softcap);
            if (k0 + lane >= see[r]) v = -INFINITY;
            const float top = fmaxf(m[r], warp_max(v)), f = expf(m[r] - top);   // every row sees key 0: finite from the first tile on
            p[r] = expf(v - top);
            l[r] = fmaf(l[r], f, warp_sum(p[r]));
            m[r] = top;
#pragma unroll
            for (int i = 0; i < NC; i++) o[r][i] *= f;
        }
        for (uint32_t j = 0; j < GA_KEYS; j++) {
            float pj[GA_RW];
#pragma unroll
            for (int r = 0; r < (int)GA_RW; r++) pj[r] = __shfl_sync(0xffffffffu, p[r], j);
            const float* c = ks + (size_t)j * ldk + s.dp + lane;
#pragma unroll
            for (int i = 0; i < NC; i++) {
                const float v = 32 * i + lane < s.vp ? c[32 * i] : 0.0f;
#pragma unroll
                for (int r = 0; r < (int)GA_RW; r++) o[r][i] = fmaf(pj[r], v, o[r][i]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < (int)GA_RW; r++) {
        const uint32_t row = r0 + warp * GA_RW + r, h = kh * group + row % group;
        if (row >= rows) break;
        OT* out = static_cast<OT*>(a.out) + (size_t)(row / group) * a.ldo + (size_t)h * s.vdim;
        const float inv = __frcp_rn(l[r]);
#pragma unroll
        for (int i = 0; i < NC; i++)
            if (32 * i + lane < s.vdim) put(out + 32 * i + lane, o[r][i] * inv);
        if (h + 1 == s.heads)   // padding up to the stride
            for (uint32_t c = s.vdim + lane; c < a.ldo - h * s.vdim; c += 32) put(out + c, 0.0f);
    }
}

template <class CT, class OT, int NC>
cudaError_t attn_inst(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    const cudaError_t err = allow_smem(grouped_attn_kernel<CT, OT, NC>, 224 * 1024, done);
    if (err != cudaSuccess) return err;
    const size_t smem = ((size_t)GA_ROWS * a.s.dp + (size_t)GA_KEYS * (a.s.dp + a.s.vp + 4)) * 4;
    if (smem > 224 * 1024) return cudaErrorInvalidValue;
    const uint32_t rows = tokens * a.s.group();
    return launch_pdl(grouped_attn_kernel<CT, OT, NC>, dim3((rows + GA_ROWS - 1) / GA_ROWS, a.s.kv_heads), dim3(256), smem, st, pdl, a, tokens);
}
template <class CT, class OT>
cudaError_t attn_type(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (a.s.vp <= 128) return attn_inst<CT, OT, 4>(a, tokens, st, pdl);
    return attn_inst<CT, OT, 16>(a, tokens, st, pdl);
}

}  // namespace

cudaError_t launch_grouped_prepare(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (a.s.dp > GROUPED_MAX_DIM || a.s.vp > GROUPED_MAX_DIM) return cudaErrorInvalidValue;
    return a.cache_bf16 ? prepare_type<bf16>(a, tokens, st, pdl) : prepare_type<float>(a, tokens, st, pdl);
}
cudaError_t launch_grouped_attn(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (a.cache_bf16) return a.act_bf16 ? attn_type<bf16, bf16>(a, tokens, st, pdl) : attn_type<bf16, float>(a, tokens, st, pdl);
    return a.act_bf16 ? cudaErrorInvalidValue : attn_type<float, float>(a, tokens, st, pdl);
}

}  // namespace alice
