// Grouped attention of many tokens over a bfloat16 cache.
//
// Scores that are bounded (unit queries and keys, or a cap) need no running maximum: exp(score) itself is summed, nothing is
// ever rescaled, and the whole of it runs as two chained products on the fifth-generation tensor cores. A CTA takes 256
// consecutive (token, head of the group) rows of one key head as two tiles of 128: warp 0 copies queries, keys and values by
// TMA, warp 1 issues the products from one thread, and four warps per tile turn its scores into weights, a row per lane. The
// weights go back into tensor memory where the scores were, as bf16 pairs (value and remainder), and are the A operand of the
// second product; while one tile's weights are made the other tile's products run. Every wait is bounded.
//
// Other sizes and unbounded scores run on attn_prefill.cuh.
#include "attn_prefill.cuh"
#include "tc_dev.cuh"

namespace alice {
namespace {

constexpr uint32_t GP_KEYS = 128, GP_ROWS = 128, GP_THREADS = 320, GP_STAGES = 2, GP_BOX = GP_ROWS * 128;
constexpr uint32_t GP_O_COL = 256;          // tensor memory: scores of the two tiles at 0 and 128, sums at 256 and 384
constexpr int KERR_ATTN_WAIT = 9;           // a wait inside the tensor-core attention
constexpr int CAP_NONE = 0, CAP_EXP = -1;   // otherwise: terms of the odd series of tanh

struct GpArgs {
    uint32_t heads, group, dp, vp, vdim, tokens, plane_rows, ldo;
    float cap2, k2;                         // CAP_NONE: k2 = scale in powers of two; CAP_EXP: cap * log2(e), 2 log2(e) scale / cap
    float series[8];                        // score in powers of two = r (series[0] + r^2 (series[1] + ...))
    const int* pos;
    const float* sink;
    bf16* out;
    int* status;
    CUtensorMap tq, tkv;                    // queries [kv_heads * rows][dp]; cache [kv_heads * plane_rows][ld]
};

using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
    f32x2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ float exp2_fast(float x) {   // |x| < 126 here
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// 32 raw scores of a row -> weights as bf16 pairs, r[0 .. 16) values and r[16 .. 32) remainders; adds them to sum. `see`: how
// many of the 32 keys the row sees (MASK).
template <int CAP, bool MASK>
__device__ __forceinline__ void weights_32(uint32_t (&r)[32], const GpArgs& a, const f32x2 (&series)[CAP > 0 ? CAP : 1], int see, f32x2 (&sum)[2]) {
    uint32_t out[32];
#pragma unroll
    for (int p = 0; p < 16; p++) {
        const float s0 = __uint_as_float(r[2 * p]), s1 = __uint_as_float(r[2 * p + 1]);
        float2 y;
        if constexpr (CAP > 0) {
            const f32x2 s = pack2(s0, s1), u = mul2(s, s);
            f32x2 t = series[CAP - 1];
#pragma unroll
            for (int i = CAP - 2; i >= 0; i--) t = fma2(u, t, series[i]);
            y = unpack2(mul2(s, t));
        } else if constexpr (CAP == CAP_EXP) {
            y = make_float2(a.cap2 * tanh_of_pow2(s0 * a.k2), a.cap2 * tanh_of_pow2(s1 * a.k2));
        } else {
            y = make_float2(s0 * a.k2, s1 * a.k2);
        }
        float x0 = exp2_fast(y.x), x1 = exp2_fast(y.y);
        if constexpr (MASK) {
            x0 = 2 * p < see ? x0 : 0.0f;
            x1 = 2 * p + 1 < see ? x1 : 0.0f;
        }
        const f32x2 x = pack2(x0, x1);
        sum[p & 1] = add2(sum[p & 1], x);
        out[p] = pack_bf16(x0, x1);
        const float2 h = bf2(out[p]);
        const float2 lo = unpack2(fma2(pack2(h.x, h.y), pack2(-1.0f, -1.0f), x));
        out[16 + p] = pack_bf16(lo.x, lo.y);
    }
#pragma unroll
    for (int i = 0; i < 32; i++) r[i] = out[i];
}

// grid (kv_heads, blocks of 256 rows)
template <int CAP>
__global__ void __launch_bounds__(GP_THREADS, 1) grouped_prefill_kernel(const __grid_constant__ GpArgs a) {
    extern __shared__ uint8_t raw[];
    __shared__ __align__(8) uint64_t q_full, k_full[GP_STAGES], k_empty[GP_STAGES], v_full[GP_STAGES], v_empty[GP_STAGES], s_full[2], p_full[2], o_full;
    __shared__ uint32_t tmem_base;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t qb = (a.dp + 63) / 64, vb = (a.vp + 63) / 64;   // boxes of 64 columns
    const uint32_t q_sm = (smem_u32(raw) + 1023u) & ~1023u, k_sm = q_sm + 2 * qb * GP_BOX, v_sm = k_sm + GP_STAGES * qb * GP_BOX;
    auto bar = [](uint64_t& b) { return smem_u32(&b); };
    if (threadIdx.x == 0) {
        mbar_init(bar(q_full), 1);
        for (uint32_t i = 0; i < GP_STAGES; i++) { mbar_init(bar(k_full[i]), 1); mbar_init(bar(k_empty[i]), 1); mbar_init(bar(v_full[i]), 1); mbar_init(bar(v_empty[i]), 1); }
        for (int i = 0; i < 2; i++) { mbar_init(bar(s_full[i]), 1); mbar_init(bar(p_full[i]), GP_ROWS); }
        mbar_init(bar(o_full), 1);
        mbar_fence_init();
        fence_proxy_async();
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base)), "n"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_base;
    pdl_launch_dependents();   // not before the tensor memory is had: a later kernel's CTA could hold it and wait for this one
    pdl_wait();

    const uint32_t p0 = (uint32_t)*a.pos, total = a.tokens * a.group, kh = blockIdx.x;
    const uint32_t r0 = (gridDim.y - 1 - blockIdx.y) * 2 * GP_ROWS, rows = min(2 * GP_ROWS, total - r0), ntile = rows > GP_ROWS ? 2 : 1;   // the longest rows first
    const uint32_t keys = p0 + (r0 + rows - 1) / a.group + 1, nt = (keys + GP_KEYS - 1) / GP_KEYS;
    if (warp == 0) {
        if (lane == 0) {
            const int qy = (int)(kh * total + r0), ky = (int)(kh * a.plane_rows);
            mbar_arrive_expect_tx(bar(q_full), ntile * qb * GP_BOX);
            for (uint32_t i = 0; i < ntile; i++)
                for (uint32_t b = 0; b < qb; b++) tma_2d(q_sm + (i * qb + b) * GP_BOX, &a.tq, (int)(b * 64), qy + (int)(i * GP_ROWS), bar(q_full));
            uint32_t k_sent = 0, v_sent = 0;
            bool ok = true;
            for (uint32_t j = 0; j < nt && ok; j++) {
                const uint32_t s = j % GP_STAGES, free = ((j / GP_STAGES) & 1) ^ 1;
                if (!(ok = mbar_wait(bar(k_empty[s]), free))) break;
                mbar_arrive_expect_tx(bar(k_full[s]), qb * GP_BOX);
                for (uint32_t b = 0; b < qb; b++) tma_2d(k_sm + (s * qb + b) * GP_BOX, &a.tkv, (int)(b * 64), ky + (int)(j * GP_KEYS), bar(k_full[s]));
                k_sent++;
                if (!(ok = mbar_wait(bar(v_empty[s]), free))) break;
                mbar_arrive_expect_tx(bar(v_full[s]), vb * GP_BOX);
                for (uint32_t b = 0; b < vb; b++) tma_2d(v_sm + (s * vb + b) * GP_BOX, &a.tkv, (int)(a.dp + b * 64), ky + (int)(j * GP_KEYS), bar(v_full[s]));
                v_sent++;
            }
            if (!ok) atomicCAS(a.status, 0, KERR_ATTN_WAIT);
            // every copy has landed before the CTA may leave
            mbar_wait(bar(q_full), 0);
            for (uint32_t j = k_sent - min(k_sent, GP_STAGES); j < k_sent; j++) mbar_wait(bar(k_full[j % GP_STAGES]), (j / GP_STAGES) & 1);
            for (uint32_t j = v_sent - min(v_sent, GP_STAGES); j < v_sent; j++) mbar_wait(bar(v_full[j % GP_STAGES]), (j / GP_STAGES) & 1);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t s_desc = mma_desc(GP_ROWS, GP_KEYS), o_desc = mma_desc(GP_ROWS, a.vp, true);
            auto scores = [&](uint32_t i, uint32_t j) {   // tile i against keys j
                const uint32_t qa = q_sm + i * qb * GP_BOX, ka = k_sm + j % GP_STAGES * qb * GP_BOX;
                for (uint32_t kk = 0; kk < a.dp / 16; kk++)
                    mma_f16(tmem + i * GP_KEYS, smem_desc(qa + kk / 4 * GP_BOX) + 2 * (kk % 4), smem_desc(ka + kk / 4 * GP_BOX) + 2 * (kk % 4), s_desc, kk > 0);
                mma_commit(bar(s_full[i]));
            };
            bool ok = mbar_wait(bar(q_full), 0) && mbar_wait(bar(k_full[0]), 0);
            if (ok) {
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                for (uint32_t i = 0; i < ntile; i++) scores(i, 0);
                mma_commit(bar(k_empty[0]));
            }
            for (uint32_t j = 0; j < nt && ok; j++) {
                const uint32_t s = j % GP_STAGES, n = (j + 1) % GP_STAGES;
                if (!(ok = mbar_wait(bar(v_full[s]), (j / GP_STAGES) & 1))) break;
                if (j + 1 < nt && !(ok = mbar_wait(bar(k_full[n]), ((j + 1) / GP_STAGES) & 1))) break;
                for (uint32_t i = 0; i < ntile && ok; i++) {
                    if (!(ok = mbar_wait(bar(p_full[i]), j & 1))) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint32_t va = v_sm + s * vb * GP_BOX, pa = tmem + i * GP_KEYS, oa = tmem + GP_O_COL + i * GP_KEYS;
                    for (uint32_t c = 0; c < GP_KEYS / 16; c++) {   // sixteen keys: their values, then their remainders
                        const uint64_t vd = smem_desc_n(va + c * 16 * 128, GP_BOX);
                        const uint32_t pc = pa + c / 2 * 32 + c % 2 * 8;
                        mma_f16_ta(oa, pc, vd, o_desc, j > 0 || c > 0);
                        mma_f16_ta(oa, pc + 16, vd, o_desc, true);
                    }
                    if (i + 1 == ntile) mma_commit(bar(v_empty[s]));
                    if (j + 1 < nt) {   // products run in the order they are issued: the weights have been read when the scores come
                        scores(i, j + 1);
                        if (i + 1 == ntile) mma_commit(bar(k_empty[n]));
                    }
                }
            }
            if (!ok) atomicCAS(a.status, 0, KERR_ATTN_WAIT);
            mma_commit(bar(o_full));
            if (!mbar_wait(bar(o_full), 0)) atomicCAS(a.status, 0, KERR_ATTN_WAIT);   // nothing runs any more when the tensor memory goes back
        }
    } else if ((warp - 2) / 4 < ntile) {
        const uint32_t i = (warp - 2) / 4, quad = warp & 3, row = r0 + i * GP_ROWS + quad * 32 + lane;
        const uint32_t see = p0 + min(row, total - 1) / a.group + 1, all_see = p0 + (r0 + i * GP_ROWS) / a.group + 1;   // keys this row sees, all rows see
        const uint32_t sa = tmem + ((quad * 32) << 16) + i * GP_KEYS;
        f32x2 series[CAP > 0 ? CAP : 1], sum[2] = {0ull, 0ull};
        if constexpr (CAP > 0)
#pragma unroll
            for (int c = 0; c < CAP; c++) series[c] = pack2(a.series[c], a.series[c]);
        bool ok = true;
        for (uint32_t j = 0; j < nt; j++) {
            ok = __all_sync(0xffffffffu, mbar_wait(bar(s_full[i]), j & 1));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            uint32_t s[2][32];
            tmem_get32(s[0], sa);
            const bool mask = (j + 1) * GP_KEYS > all_see;
#pragma unroll
            for (int c = 0; c < (int)GP_KEYS / 32; c++) {
                tmem_got32(s[c & 1]);
                if (c + 1 < (int)GP_KEYS / 32) tmem_get32(s[(c + 1) & 1], sa + (c + 1) * 32);
                if (mask) weights_32<CAP, true>(s[c & 1], a, series, (int)see - (int)(j * GP_KEYS + c * 32), sum);
                else weights_32<CAP, false>(s[c & 1], a, series, 32, sum);
                tmem_put32(sa + c * 32, s[c & 1]);
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(bar(p_full[i]));
        }
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait(bar(o_full), 0));
        if (!ok) {
            if (lane == 0) atomicCAS(a.status, 0, KERR_ATTN_WAIT);
        } else {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t h = kh * a.group + row % a.group;
            const float2 l0 = unpack2(sum[0]), l1 = unpack2(sum[1]);
            float inv = 0.0f;
            bf16* out = nullptr;
            if (row < total) {
                inv = __frcp_rn((l0.x + l0.y) + (l1.x + l1.y) + expf(a.sink[h]));   // an infinite sink leaves zeros
                out = a.out + (size_t)(row / a.group) * a.ldo + (size_t)h * a.vdim;
            }
            for (uint32_t c = 0; c < a.vdim; c += 32) {
                float v[32];
                __syncwarp();
                tmem_ld32(v, tmem + ((quad * 32) << 16) + GP_O_COL + i * GP_KEYS + c);
                if (out) {
                    if (a.vdim % 8 == 0) {
#pragma unroll
                        for (int e = 0; e < 32; e += 8)
                            if (c + e < a.vdim)
                                *reinterpret_cast<uint4*>(out + c + e) = make_uint4(pack_bf16(v[e] * inv, v[e + 1] * inv), pack_bf16(v[e + 2] * inv, v[e + 3] * inv),
                                                                                    pack_bf16(v[e + 4] * inv, v[e + 5] * inv), pack_bf16(v[e + 6] * inv, v[e + 7] * inv));
                    } else {
#pragma unroll
                        for (int e = 0; e < 32; e++)
                            if (c + e < a.vdim) put(out + c + e, v[e] * inv);
                    }
                }
            }
            if (out && h + 1 == a.heads)   // padding up to the stride
                for (uint32_t c = a.vdim; c < a.ldo - h * a.vdim; c++) put(out + c, 0.0f);
        }
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    }
    __syncwarp();
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(512));
    }
}

template <int CAP>
cudaError_t prefill_inst(const GpArgs& a, uint32_t kv_heads, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    const cudaError_t err = allow_smem(grouped_prefill_kernel<CAP>, 200 * 1024, done);
    if (err != cudaSuccess) return err;
    const size_t boxes = (size_t)(2 + GP_STAGES) * ((a.dp + 63) / 64) + GP_STAGES * ((a.vp + 63) / 64);
    const size_t smem = std::max<size_t>(boxes * GP_BOX + 1024, 120 * 1024);   // one CTA per SM: each takes all of the tensor memory
    return launch_pdl(grouped_prefill_kernel<CAP>, dim3(kv_heads, (a.tokens * a.group + 2 * GP_ROWS - 1) / (2 * GP_ROWS)), dim3(GP_THREADS), smem, st, pdl, a);
}

bool tc_fits(const GroupedArgs& a) { return a.s.dp <= 128 && a.s.vp <= 128 && a.bounded; }

cudaError_t prefill_tc(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (!encode_fn()) return cudaErrorNotSupported;
    const GroupedShape& z = a.s;
    constexpr double LOG2E = 1.4426950408889634;
    GpArgs g = {};
    g.heads = z.heads; g.group = z.group(); g.dp = z.dp; g.vp = z.vp; g.vdim = z.vdim; g.tokens = tokens; g.plane_rows = a.plane_rows; g.ldo = a.ldo;
    g.pos = a.pos; g.sink = a.sink; g.out = static_cast<bf16*>(a.out); g.status = a.status;
    if (!tile_map(&g.tq, a.q, z.heads * tokens, z.dp, z.dp, GP_ROWS) || !tile_map(&g.tkv, a.cache, z.kv_heads * a.plane_rows, z.ld(), z.ld(), GP_KEYS))
        return cudaErrorInvalidValue;
    if (z.softcap <= 0.0f) {
        g.k2 = (float)(z.scale * LOG2E);
        return prefill_inst<CAP_NONE>(g, z.kv_heads, st, pdl);
    }
    g.cap2 = (float)(z.softcap * LOG2E);
    g.k2 = (float)(2.0 * LOG2E * z.scale / z.softcap);
    // arguments of tanh up to `most`: the odd series to a few parts in 1e7 of its value, with cap and scale multiplied in
    static const double tanh_series[8] = {1.0, -1.0 / 3, 2.0 / 15, -17.0 / 315, 62.0 / 2835, -1382.0 / 155925, 21844.0 / 6081075, -929569.0 / 638512875};
    const double most = z.unit_qk ? 1.01 * std::fabs(z.scale) * z.dim / z.softcap : INFINITY, f = z.scale / z.softcap;
    for (int i = 0; i < 8; i++) g.series[i] = (float)(tanh_series[i] * z.softcap * LOG2E * std::pow(f, 2 * i + 1));
    if (most <= 0.35) return prefill_inst<5>(g, z.kv_heads, st, pdl);
    if (most <= 0.6) return prefill_inst<8>(g, z.kv_heads, st, pdl);
    return prefill_inst<CAP_EXP>(g, z.kv_heads, st, pdl);
}

cudaError_t prefill_sync(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const GroupedShape& z = a.s;
    const auto* cache = static_cast<const bf16*>(a.cache);
    PrefillArgs p;
    p.heads = z.heads; p.group = z.group(); p.vdim = z.vdim; p.v_cols = z.vp; p.pos = a.pos; p.sink = a.sink; p.scale = z.scale; p.softcap = z.softcap;
    p.q = static_cast<const bf16*>(a.q); p.q_row = (size_t)z.group() * z.dp; p.q_group = tokens * p.q_row; p.k1 = cache; p.k1_cols = z.dp; p.v = cache + z.dp;
    p.k1_row = p.v_row = z.ld(); p.k1_head = p.v_head = (size_t)a.plane_rows * z.ld();
    p.out = static_cast<bf16*>(a.out); p.ldo = a.ldo;
    return launch_attn_prefill<true>(p, tokens, st, pdl);
}

}  // namespace

cudaError_t launch_grouped_prefill(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (!grouped_tiled_fits(a.s) || !a.cache_bf16 || !a.act_bf16) return cudaErrorInvalidValue;
    return tc_fits(a) ? prefill_tc(a, tokens, st, pdl) : prefill_sync(a, tokens, st, pdl);
}

}  // namespace alice
