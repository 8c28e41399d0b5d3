// Delta rule with one decay per key channel. Per head, with a state S [dim][vdim] kept in f32:
//   S <- g * S (rows);  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
// Columns of S never meet, so the state is cut by columns. Many tokens go in blocks of W = 16. With G_t the product of the
// decays up to token t of a block, and P_st that of the decays after s up to t,
//   A_ts = sum_d k_t k_s P_st (s < t),  B_ts = sum_d q_t k_s P_st (s <= t),
// the block's writes solve (I + diag(beta) A) u = diag(beta) (v - S^T (G k)), and
//   o_t = S^T (G_t q_t) + sum_s B_ts u_s,   S <- G_W S + sum_s (P_sW k_s) u_s^T.
// A, B and the inverse depend on the projections only and are made for all blocks at once; what remains on the path from
// block to block are three small products per block, in f32. Decays enter as products, never as quotients.
#include "dense_dev.cuh"
#include "mixers.cuh"

namespace alice {
namespace {

// Inputs of the convolution before the tokens at hand, and where those of the next call go.
__device__ __forceinline__ const float* conv_before(const DeltaArgs& a) {
    return a.conv_state + (size_t)(*a.pos & 1) * (a.s.taps - 1) * a.s.conv_cols;
}
__device__ __forceinline__ float* conv_after(const DeltaArgs& a, uint32_t tokens) {
    return a.conv_state + (size_t)((*a.pos + (int)tokens) & 1) * (a.s.taps - 1) * a.s.conv_cols;
}
// Convolution and silu of channel c at token t.
__device__ __forceinline__ float conv_silu(const DeltaArgs& a, const float* before, int t, uint32_t c) {
    const int taps = (int)a.s.taps;
    const float* w = a.conv_w + c;
    float v = 0.0f;
    for (int j = 0; j < taps; j++) {
        const int s = t - (taps - 1 - j);
        v = fmaf(w[(size_t)j * a.s.conv_cols], s >= 0 ? a.y[(size_t)s * a.ldy + c] : before[(size_t)(taps - 1 + s) * a.s.conv_cols + c], v);
    }
    return silu_ref(v);
}
// Inputs of channel c that the next call needs: the last taps - 1 of [before; the tokens at hand].
__device__ __forceinline__ void conv_keep(const DeltaArgs& a, const float* before, float* after, uint32_t tokens, uint32_t c) {
    const uint32_t keep = a.s.taps - 1;
    for (uint32_t j = 0; j < keep; j++) {
        const uint32_t i = tokens + j;
        after[(size_t)j * a.s.conv_cols + c] = i < keep ? before[(size_t)i * a.s.conv_cols + c] : a.y[(size_t)(i - keep) * a.ldy + c];
    }
}

constexpr int PREP_TOKENS = 8;   // consecutive tokens of a warp
// Convolution and silu of channel c for PREP_TOKENS tokens from t0 on. TAPS > 0: the number of taps, known when compiled.
template <int TAPS>
__device__ __forceinline__ void conv_run(const DeltaArgs& a, const float* before, int t0, uint32_t tokens, uint32_t c, float (&out)[PREP_TOKENS]) {
    if constexpr (TAPS == 0) {
#pragma unroll
        for (int j = 0; j < PREP_TOKENS; j++) out[j] = (uint32_t)(t0 + j) < tokens ? conv_silu(a, before, t0 + j, c) : 0.0f;
    } else {
        float w[TAPS], x[PREP_TOKENS + TAPS - 1];
#pragma unroll
        for (int j = 0; j < TAPS; j++) w[j] = a.conv_w[(size_t)j * a.s.conv_cols + c];
#pragma unroll
        for (int j = 0; j < PREP_TOKENS + TAPS - 1; j++) {
            const int s = t0 + j - (TAPS - 1);
            x[j] = s < 0 ? before[(size_t)(TAPS - 1 + s) * a.s.conv_cols + c] : (uint32_t)s < tokens ? a.y[(size_t)s * a.ldy + c] : 0.0f;
        }
#pragma unroll
        for (int j = 0; j < PREP_TOKENS; j++) {
            float v = 0.0f;
#pragma unroll
            for (int i = 0; i < TAPS; i++) v = fmaf(w[i], x[j + i], v);
            out[j] = silu_ref(v);
        }
    }
}

// One warp per head (key heads, then value heads) and PREP_TOKENS tokens: convolution, silu, unit vectors, step size.
template <int TAPS, int N>   // N: 32-channel groups of a padded key head
__global__ void __launch_bounds__(128) delta_prepare_kernel(const __grid_constant__ DeltaArgs a, uint32_t tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const DeltaShape& s = a.s;
    const uint32_t lane = threadIdx.x & 31, t0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * PREP_TOKENS, i = blockIdx.y;
    if (t0 >= tokens) return;
    const uint32_t n = min(tokens - t0, (uint32_t)PREP_TOKENS);
    const float* before = conv_before(a);
    if (i < s.kv_heads) {
#pragma unroll 1
        for (int which = 0; which < 2; which++) {   // q, then k
            const uint32_t off = (which ? s.off_k : s.off_q) + i * s.dim;
            float v[N][PREP_TOKENS], ss[PREP_TOKENS] = {};
#pragma unroll
            for (int g = 0; g < N; g++) {
                const uint32_t d = lane + 32 * g;
                if (d < s.dim) {
                    conv_run<TAPS>(a, before, (int)t0, tokens, off + d, v[g]);
                } else {
#pragma unroll
                    for (int j = 0; j < PREP_TOKENS; j++) v[g][j] = 0.0f;
                }
#pragma unroll
                for (int j = 0; j < PREP_TOKENS; j++) ss[j] = fmaf(v[g][j], v[g][j], ss[j]);
            }
            float* out = (which ? a.kn : a.qn) + ((size_t)t0 * s.kv_heads + i) * s.dp;
#pragma unroll
            for (int j = 0; j < PREP_TOKENS; j++) {
                float inv = __frcp_rn(__fsqrt_rn(warp_sum(ss[j]) + 1e-6f));
                if (which == 0) inv *= __frcp_rn(__fsqrt_rn((float)s.dim));
                if ((uint32_t)j < n)
#pragma unroll
                    for (int g = 0; g < N; g++) out[(size_t)j * s.kv_heads * s.dp + lane + 32 * g] = v[g][j] * inv;
            }
        }
    } else {
        const uint32_t h = i - s.kv_heads;
        for (uint32_t d = lane; d < s.vp; d += 32) {
            float v[PREP_TOKENS] = {};
            if (d < s.vdim) conv_run<TAPS>(a, before, (int)t0, tokens, s.off_v + h * s.vdim + d, v);
#pragma unroll
            for (int j = 0; j < PREP_TOKENS; j++)
                if ((uint32_t)j < n) a.v[((size_t)(t0 + j) * s.heads + h) * s.vp + d] = v[j];
        }
        if (lane < n) a.beta[(size_t)(t0 + lane) * s.heads + h] = sigmoid_f(a.y[(size_t)(t0 + lane) * a.ldy + s.off_b + h]);
    }
}

// The two halves of the convolution state differ unless an even number of tokens passed: then this call reads and writes the
// same half. A thread owns its channel, reads ahead of what it overwrites, and runs after all other readers.
__global__ void __launch_bounds__(256) conv_tail_kernel(const __grid_constant__ DeltaArgs a, uint32_t tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t c = blockIdx.x * 256 + threadIdx.x;
    if (c < a.s.conv_cols) conv_keep(a, conv_before(a), conv_after(a, tokens), tokens, c);
}

constexpr int SCAN_COLS = 32;   // columns per CTA of a single token's step
constexpr int W = 16;           // tokens per block

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool ok = true) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(ok ? 16u : 0u) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// grid (blocks, heads): inv = (I + diag(beta) A)^-1 diag(beta) and B of every block, [W][W] each. Sixteen lanes share a key s
// and walk its decayed form along the later tokens.
template <int DP>
__global__ void __launch_bounds__(256) delta_pairs_kernel(const __grid_constant__ DeltaArgs a, uint32_t tokens) {
    constexpr int ED = DP / 16;
    extern __shared__ __align__(16) float sm[];
    float *k = sm, *q = k + W * DP, *g = q + W * DP;
    __shared__ float A[W][W + 1], B[W][W + 1], beta[W];
    const DeltaShape& s = a.s;
    const uint32_t tid = threadIdx.x, h = blockIdx.y, kh = h / (s.heads / s.kv_heads), t0 = blockIdx.x * W, n = min(tokens - t0, (uint32_t)W);
    pdl_launch_dependents();
    pdl_wait();
    for (uint32_t i = tid; i < W * DP / 4; i += 256) {
        const uint32_t t = i / (DP / 4), d = i % (DP / 4) * 4;
        float4 kk = make_float4(0.f, 0.f, 0.f, 0.f), qq = kk, gg = kk;
        if (t < n) {
            const size_t ko = ((size_t)(t0 + t) * s.kv_heads + kh) * DP + d;
            kk = *reinterpret_cast<const float4*>(a.kn + ko);
            qq = *reinterpret_cast<const float4*>(a.qn + ko);
            gg = *reinterpret_cast<const float4*>(a.g + ((size_t)(t0 + t) * s.heads + h) * DP + d);
        }
        *reinterpret_cast<float4*>(k + t * DP + d) = kk;
        *reinterpret_cast<float4*>(q + t * DP + d) = qq;
        *reinterpret_cast<float4*>(g + t * DP + d) = gg;
    }
    if (tid < W) beta[tid] = tid < n ? a.beta[(size_t)(t0 + tid) * s.heads + h] : 0.0f;
    A[tid / W][tid % W] = 0.0f;
    B[tid / W][tid % W] = 0.0f;
    __syncthreads();
    const uint32_t ks = tid >> 4, l = tid & 15;
    float p[ED];
#pragma unroll
    for (int e = 0; e < ED; e++) p[e] = k[ks * DP + (e / 4) * 64 + l * 4 + e % 4];
    for (uint32_t t = (tid >> 5) * 2; t < W; t++) {   // the first of the warp's two keys
        float x = 0.0f, y = 0.0f;
#pragma unroll
        for (int e = 0; e < ED; e += 4) {
            const uint32_t o = t * DP + e * 16 + l * 4;
            const float4 kk = *reinterpret_cast<const float4*>(k + o), qq = *reinterpret_cast<const float4*>(q + o), gg = *reinterpret_cast<const float4*>(g + o);
            if (t > ks) { p[e] *= gg.x; p[e + 1] *= gg.y; p[e + 2] *= gg.z; p[e + 3] *= gg.w; }
            x = fmaf(p[e], kk.x, x); x = fmaf(p[e + 1], kk.y, x); x = fmaf(p[e + 2], kk.z, x); x = fmaf(p[e + 3], kk.w, x);
            y = fmaf(p[e], qq.x, y); y = fmaf(p[e + 1], qq.y, y); y = fmaf(p[e + 2], qq.z, y); y = fmaf(p[e + 3], qq.w, y);
        }
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) {
            x += __shfl_xor_sync(0xffffffffu, x, o);
            y += __shfl_xor_sync(0xffffffffu, y, o);
        }
        if (l == 0 && t >= ks) {
            if (t > ks) A[t][ks] = beta[t] * x;
            B[t][ks] = y;
        }
    }
    __syncthreads();
    const size_t o = ((size_t)blockIdx.x * s.heads + h) * W * W;
    a.pair_b[o + tid] = B[tid / W][tid % W];
    if (tid < W) {   // column tid of the inverse by forward substitution
        float x[W];
#pragma unroll
        for (int t = 0; t < W; t++) {
            float v = t == (int)tid ? beta[t] : 0.0f;
#pragma unroll
            for (int j = 0; j < t; j++) v = fmaf(-A[t][j], x[j], v);
            x[t] = v;
        }
#pragma unroll
        for (int t = 0; t < W; t++) a.pair_inv[o + t * W + tid] = x[t];
    }
}

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;"
        : "=l"(*reinterpret_cast<unsigned long long*>(&d))
        : "l"(*reinterpret_cast<const unsigned long long*>(&a)), "l"(*reinterpret_cast<const unsigned long long*>(&b)),
          "l"(*reinterpret_cast<const unsigned long long*>(&c)));
    return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("mul.rn.f32x2 %0, %1, %2;"
        : "=l"(*reinterpret_cast<unsigned long long*>(&d))
        : "l"(*reinterpret_cast<const unsigned long long*>(&a)), "l"(*reinterpret_cast<const unsigned long long*>(&b)));
    return d;
}

// Sums 64 values over each half-warp; lane l of it is left with those of index 4 l .. 4 l + 3.
__device__ __forceinline__ float4 reduce64(float (&v)[64], uint32_t lane) {
#pragma unroll
    for (int half = 32, o = 8; o > 0; half >>= 1, o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int i = 0; i < half; i++) {
            const float send = up ? v[i] : v[i + half], keep = up ? v[i + half] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
    return make_float4(v[0], v[1], v[2], v[3]);
}

template <int DP, int NW>
struct ScanStage {
    float k[W][DP], q[W][DP], g[W][DP], v[W][8 * NW], inv[W][W], b[W][W];
};
template <int DP, int NW>
struct ScanSmem {
    ScanStage<DP, NW> st[2];
    float end[DP];                 // decay over the whole block
    float w[W][8 * NW];            // v - S^T (G k)
    float y[W][8 * NW];            // S^T (G q)
    float2 u[W][8 * NW];           // writes, twice each
};

template <int DP, int NW>
__device__ __forceinline__ void scan_fetch(ScanStage<DP, NW>& st, const DeltaArgs& a, uint32_t t0, uint32_t n, uint32_t h, uint32_t kh, uint32_t c0) {
    const DeltaShape& s = a.s;
    for (uint32_t i = threadIdx.x; i < W * DP / 4; i += NW * 32) {
        const uint32_t j = i / (DP / 4), d = i % (DP / 4) * 4, t = t0 + min(j, n - 1);
        const size_t ko = ((size_t)t * s.kv_heads + kh) * DP + d;
        cp_async16(&st.k[j][d], a.kn + ko, j < n);
        cp_async16(&st.q[j][d], a.qn + ko, j < n);
        cp_async16(&st.g[j][d], a.g + ((size_t)t * s.heads + h) * DP + d, j < n);
    }
    for (uint32_t i = threadIdx.x; i < W * 2 * NW; i += NW * 32) {
        const uint32_t j = i / (2 * NW), d = i % (2 * NW) * 4, t = t0 + min(j, n - 1);
        cp_async16(&st.v[j][d], a.v + ((size_t)t * s.heads + h) * s.vp + c0 + d, j < n);
    }
    const size_t o = ((size_t)(t0 / W) * s.heads + h) * W * W;
    for (uint32_t i = threadIdx.x; i < W * W / 4; i += NW * 32) {
        cp_async16(&st.inv[0][0] + i * 4, a.pair_inv + o + i * 4);
        cp_async16(&st.b[0][0] + i * 4, a.pair_b + o + i * 4);
    }
}

// grid (vp / (8 NW), heads), NW warps; a warp owns eight columns of the state, four per half-warp, a lane DP / 16 of their rows
// (register pairs).
template <int DP, int NW>
__global__ void __launch_bounds__(NW * 32) delta_scan_kernel(const __grid_constant__ DeltaArgs a, uint32_t tokens) {
    constexpr int EL = DP / 16, NP = EL / 2, NC = EL / 4, COLS = 8 * NW;   // rows per lane, in NC runs of four
    extern __shared__ __align__(16) uint8_t raw[];
    auto& sm = *reinterpret_cast<ScanSmem<DP, NW>*>(raw);
    const DeltaShape& s = a.s;
    const uint32_t tid = threadIdx.x, lane = tid & 31, dg = lane & 15, warp = tid >> 5, h = blockIdx.y, kh = h / (s.heads / s.kv_heads), c0 = blockIdx.x * COLS;
    const uint32_t cw = warp * 8, cl = cw + (lane >> 4) * 4;   // first column of the warp, of the lane
    float* sp = a.state + ((size_t)h * s.vp + c0 + cl) * DP + dg * 4;
    pdl_launch_dependents();
    pdl_wait();
    auto rows = [](const float* p, float2 (&r)[NP]) {   // this lane's rows of a [DP] vector
#pragma unroll
        for (int i = 0; i < NC; i++) {
            const float4 f = *reinterpret_cast<const float4*>(p + i * 64);
            r[2 * i] = make_float2(f.x, f.y); r[2 * i + 1] = make_float2(f.z, f.w);
        }
    };
    float2 S[4][NP];
#pragma unroll
    for (int c = 0; c < 4; c++) rows(sp + c * DP, S[c]);
    const uint32_t nblk = (tokens + W - 1) / W;
    scan_fetch<DP, NW>(sm.st[0], a, 0, min(tokens, (uint32_t)W), h, kh, c0);
    cp_commit();
    for (uint32_t blk = 0; blk < nblk; blk++) {
        const uint32_t t0 = blk * W, n = min(tokens - t0, (uint32_t)W);
        ScanStage<DP, NW>& st = sm.st[blk & 1];
        if (blk + 1 < nblk) scan_fetch<DP, NW>(sm.st[(blk + 1) & 1], a, t0 + W, min(tokens - t0 - W, (uint32_t)W), h, kh, c0);
        cp_commit();
        cp_wait<1>();
        __syncthreads();
        // in place: k -> G k, q -> G q, g -> (decays after s) k_s; absent tokens have k = q = 0 and decay 1
        for (uint32_t d = tid; d < DP; d += NW * 32) {
            float k[W], g[W], p = 1.0f;
#pragma unroll
            for (int t = 0; t < W; t++) {
                k[t] = st.k[t][d];
                g[t] = (uint32_t)t < n ? st.g[t][d] : 1.0f;
                p *= g[t];
                st.k[t][d] = p * k[t];
                st.q[t][d] *= p;
            }
            sm.end[d] = p;
            p = 1.0f;
#pragma unroll
            for (int t = W - 1; t >= 0; t--) {
                st.g[t][d] = p * k[t];
                p *= g[t];
            }
        }
        __syncthreads();
#pragma unroll 1
        for (int pass = 0; pass < 2; pass++) {   // S^T (G k), then S^T (G q)
            float v[64];
#pragma unroll
            for (int t = 0; t < W; t++) {
                float2 x[NP];
                rows((pass ? st.q[t] : st.k[t]) + dg * 4, x);
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    float2 acc = mul2(x[0], S[c][0]);
#pragma unroll
                    for (int i = 1; i < NP; i++) acc = fma2(x[i], S[c][i], acc);
                    v[t * 4 + c] = acc.x + acc.y;
                }
            }
            const float4 r = reduce64(v, lane);   // token dg, the lane's four columns
            if (pass == 0) {
                const float4 x = *reinterpret_cast<const float4*>(&st.v[dg][cl]);
                *reinterpret_cast<float4*>(&sm.w[dg][cl]) = make_float4(x.x - r.x, x.y - r.y, x.z - r.z, x.w - r.w);
            } else {
                *reinterpret_cast<float4*>(&sm.y[dg][cl]) = r;
            }
        }
        __syncwarp();   // from here to the end of the block a warp works on its own columns only
        {
            const uint32_t c = cw + (lane & 7), tl = lane >> 3;   // tokens tl, tl + 4, tl + 8, tl + 12 of one column
            float u[4] = {};
#pragma unroll
            for (int j = 0; j < W; j += 4) {
                const float w0 = sm.w[j][c], w1 = sm.w[j + 1][c], w2 = sm.w[j + 2][c], w3 = sm.w[j + 3][c];
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const float4 m = *reinterpret_cast<const float4*>(&st.inv[tl + 4 * i][j]);
                    u[i] = fmaf(m.x, w0, u[i]); u[i] = fmaf(m.y, w1, u[i]); u[i] = fmaf(m.z, w2, u[i]); u[i] = fmaf(m.w, w3, u[i]);
                }
            }
            float o[4];
#pragma unroll
            for (int i = 0; i < 4; i++) {
                sm.u[tl + 4 * i][c] = make_float2(u[i], u[i]);
                o[i] = sm.y[tl + 4 * i][c];
            }
            __syncwarp();
#pragma unroll
            for (int j = 0; j < W; j += 4) {
                const float w0 = sm.u[j][c].x, w1 = sm.u[j + 1][c].x, w2 = sm.u[j + 2][c].x, w3 = sm.u[j + 3][c].x;
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const float4 m = *reinterpret_cast<const float4*>(&st.b[tl + 4 * i][j]);
                    o[i] = fmaf(m.x, w0, o[i]); o[i] = fmaf(m.y, w1, o[i]); o[i] = fmaf(m.z, w2, o[i]); o[i] = fmaf(m.w, w3, o[i]);
                }
            }
            if (c0 + c < s.vdim)
#pragma unroll
                for (int i = 0; i < 4; i++)
                    if (tl + 4 * i < n) a.o[((size_t)(t0 + tl + 4 * i) * s.heads + h) * s.vdim + c0 + c] = o[i];
        }
        float2 e[NP];
        rows(sm.end + dg * 4, e);
#pragma unroll
        for (int c = 0; c < 4; c++)
#pragma unroll
            for (int i = 0; i < NP; i++) S[c][i] = mul2(e[i], S[c][i]);
#pragma unroll 4
        for (int t = 0; t < W; t++) {
            float2 x[NP];
            rows(st.g[t] + dg * 4, x);
#pragma unroll
            for (int c = 0; c < 4; c++) {
                const float2 u = sm.u[t][cl + c];
#pragma unroll
                for (int i = 0; i < NP; i++) S[c][i] = fma2(x[i], u, S[c][i]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < 4; c++)
#pragma unroll
        for (int i = 0; i < NC; i++) {
            *reinterpret_cast<float4*>(sp + c * DP + i * 64) = make_float4(S[c][2 * i].x, S[c][2 * i].y, S[c][2 * i + 1].x, S[c][2 * i + 1].y);
        }
}

// One warp per (token, head): root-mean-square norm over vdim, weight, gate.
template <class OT>
__global__ void __launch_bounds__(256) delta_out_kernel(const __grid_constant__ DeltaArgs a, uint32_t tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const DeltaShape& s = a.s;
    const uint32_t lane = threadIdx.x & 31;
    const size_t task = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (task >= (size_t)tokens * s.heads) return;
    const uint32_t t = (uint32_t)(task / s.heads), h = (uint32_t)(task % s.heads);
    const float* o = a.o + task * s.vdim;
    const float* gate = a.gate + task * s.vdim;
    float q = 0.0f;
    for (uint32_t d = lane; d < s.vdim; d += 32) q = fmaf(o[d], o[d], q);
    q = warp_sum(q);
    const float inv = __frcp_rn(__fsqrt_rn(q / (float)s.vdim + a.eps));
    OT* out = static_cast<OT*>(a.out) + (size_t)t * a.ldo + (size_t)h * s.vdim;
    for (uint32_t d = lane; d < s.vdim; d += 32) put(out + d, o[d] * inv * a.norm_w[d] * gate[d]);
    if (h + 1 == s.heads)   // padding up to the stride
        for (uint32_t d = s.vdim + lane; d < a.ldo - h * s.vdim; d += 32) put(out + d, 0.0f);
}

// One token. A cluster of vp / 32 CTAs per head, each with 32 columns of the state (eight lanes a column); the head's
// convolutions, decays and step size are worked out by every CTA for itself, the norm over vdim joins them.
template <int E>
__global__ void __launch_bounds__(256, 2) delta_step_kernel(const __grid_constant__ DeltaStepArgs a) {
    constexpr uint32_t DP = 8 * E;
    __shared__ __align__(16) float q[DP], k[DP], g[DP], v[SCAN_COLS], gate[SCAN_COLS], os[SCAN_COLS], red[8];
    extern __shared__ __align__(16) float low[];   // low-rank inputs of the decay and of the gate
    __shared__ float part[8];                      // one partial sum of squares per CTA of the cluster
    const DeltaArgs& d = a.d;
    const DeltaShape& s = d.s;
    const uint32_t ncta = s.vp / SCAN_COLS, h = blockIdx.x / ncta, rank = blockIdx.x % ncta, c0 = rank * SCAN_COLS, kh = h / (s.heads / s.kv_heads);
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, l = lane & 7, col = warp * 4 + (lane >> 3);
    float* sp = d.state + ((size_t)h * s.vp + c0 + col) * DP + l * 4;
    const bf16* wa = a.a2.w + (size_t)h * DP * a.a2.k;
    const bf16* wg = a.g2.w + ((size_t)h * s.vdim + c0) * a.g2.k;
    const uint32_t vrows = min((uint32_t)SCAN_COLS, s.vdim - c0);
    pdl_launch_dependents();
    asm volatile("barrier.cluster.arrive.relaxed;" ::: "memory");   // every CTA of the cluster runs before one writes to another
#pragma unroll
    for (int e = 0; e < E; e += 4) if (l == 0) prefetch_l2(sp + e * 8);
    for (uint32_t i = tid; i < DP * (a.a2.k / 64); i += 256) prefetch_l2(wa + (size_t)i * 64);
    for (uint32_t i = tid; i < vrows * (a.g2.k / 64); i += 256) prefetch_l2(wg + (size_t)i * 64);
    for (uint32_t j = 0; j < 3 * s.taps - 2; j++) {   // the taps, and both halves of the convolution state
        const float* b = j < s.taps ? d.conv_w + (size_t)j * s.conv_cols : d.conv_state + (size_t)(j - s.taps) * s.conv_cols;
        if (tid < s.dim && tid % 32 == 0) { prefetch_l2(b + s.off_q + kh * s.dim + tid); prefetch_l2(b + s.off_k + kh * s.dim + tid); }
        if (tid == 0) prefetch_l2(b + s.off_v + h * s.vdim + c0);
    }
    if (tid < DP && tid % 32 == 0) prefetch_l2(a.dt_bias + (size_t)h * DP + tid);
    pdl_wait();
    const float* before = conv_before(d);
    float S[E];
#pragma unroll
    for (int e = 0; e < E; e += 4) {
        const float4 f = *reinterpret_cast<const float4*>(sp + e * 8);
        S[e] = f.x; S[e + 1] = f.y; S[e + 2] = f.z; S[e + 3] = f.w;
    }
    for (uint32_t i = tid; i < a.a2.k; i += 256) low[i] = d.y[a.off_a + i];
    for (uint32_t i = tid; i < a.g2.k; i += 256) low[a.a2.k + i] = d.y[a.off_g + i];
    const float qv = tid < s.dim ? conv_silu(d, before, 0, s.off_q + kh * s.dim + tid) : 0.0f;
    const float kv = tid < s.dim ? conv_silu(d, before, 0, s.off_k + kh * s.dim + tid) : 0.0f;
    const float sq = block_sum<8>(qv * qv, red), sk = block_sum<8>(kv * kv, red);   // also publishes `low`
    if (tid < DP) {
        q[tid] = qv * __frcp_rn(__fsqrt_rn(sq + 1e-6f)) * __frcp_rn(__fsqrt_rn((float)s.dim));
        k[tid] = kv * __frcp_rn(__fsqrt_rn(sk + 1e-6f));
    }
    if (tid < SCAN_COLS) v[tid] = c0 + tid < s.vdim ? conv_silu(d, before, 0, s.off_v + h * s.vdim + c0 + tid) : 0.0f;
    const float beta = sigmoid_f(d.y[s.off_b + h]), rate = expf(a.a_log[h]);
    // low-rank projections: sixteen lanes a row, all rows of a lane group in flight at once
    const uint32_t hw = tid >> 4, hl = tid & 15;
    constexpr int ND = DP / 16;
    float acc[ND + 2];
#pragma unroll
    for (int i = 0; i < ND + 2; i++) acc[i] = 0.0f;
    for (uint32_t c = hl * 8; c < a.a2.k; c += 128) {
        const float4 x0 = *reinterpret_cast<const float4*>(low + c), x1 = *reinterpret_cast<const float4*>(low + c + 4);
#pragma unroll
        for (int i = 0; i < ND; i++) acc[i] = dot8(__ldg(reinterpret_cast<const uint4*>(wa + (size_t)(hw + 16 * i) * a.a2.k + c)), x0, x1, acc[i]);
    }
    for (uint32_t c = hl * 8; c < a.g2.k; c += 128) {
        const float4 x0 = *reinterpret_cast<const float4*>(low + a.a2.k + c), x1 = *reinterpret_cast<const float4*>(low + a.a2.k + c + 4);
#pragma unroll
        for (int i = 0; i < 2; i++)
            acc[ND + i] = dot8(__ldg(reinterpret_cast<const uint4*>(wg + (size_t)min(hw + 16 * i, vrows - 1) * a.g2.k + c)), x0, x1, acc[ND + i]);
    }
#pragma unroll
    for (int i = 0; i < ND + 2; i++) {
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], o);
        const uint32_t row = hw + 16 * (i < ND ? i : i - ND);
        if (hl == 0) {
            if (i < ND) g[row] = expf(-rate * softplus_f(acc[i] + a.dt_bias[(size_t)h * DP + row]));
            else gate[row] = sigmoid_f(acc[i]);
        }
    }
    __syncthreads();
    float dk = 0.0f, dq = 0.0f, kq = 0.0f;
#pragma unroll
    for (int e = 0; e < E; e++) {
        const uint32_t i = (e / 4) * 32 + l * 4 + e % 4;
        S[e] *= g[i];
        dk = fmaf(S[e], k[i], dk);
        dq = fmaf(S[e], q[i], dq);
        kq = fmaf(k[i], q[i], kq);
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
        dk += __shfl_xor_sync(0xffffffffu, dk, o);
        dq += __shfl_xor_sync(0xffffffffu, dq, o);
        kq += __shfl_xor_sync(0xffffffffu, kq, o);
    }
    const float u = beta * (v[col] - dk);
#pragma unroll
    for (int e = 0; e < E; e += 4) {
        const uint32_t i = e * 8 + l * 4;
        *reinterpret_cast<float4*>(sp + e * 8) = make_float4(fmaf(k[i], u, S[e]), fmaf(k[i + 1], u, S[e + 1]), fmaf(k[i + 2], u, S[e + 2]), fmaf(k[i + 3], u, S[e + 3]));
    }
    if (l == 0) os[col] = fmaf(kq, u, dq);
    __syncthreads();
    asm volatile("barrier.cluster.wait;" ::: "memory");
    float ss = 0.0f;
    if (warp == 0) {
        ss = warp_sum(lane < vrows ? os[lane] * os[lane] : 0.0f);
        if (lane < ncta) {   // the slice's sum of squares into every CTA of the cluster
            uint32_t dst;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"(smem_u32(&part[rank])), "r"(lane));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(ss) : "memory");
        }
    }
    asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory");
    if (tid < vrows) {
        float tot = 0.0f;
        for (uint32_t i = 0; i < ncta; i++) tot += part[i];
        const float inv = __frcp_rn(__fsqrt_rn(tot / (float)s.vdim + d.eps));
        static_cast<float*>(d.out)[(size_t)h * s.vdim + c0 + tid] = os[tid] * inv * d.norm_w[c0 + tid] * gate[tid];
    }
    // what the next token's convolution needs: a head's own value columns, and the key head's channels once per key head
    float* after = conv_after(d, 1);
    if (tid < vrows) conv_keep(d, before, after, 1, s.off_v + h * s.vdim + c0 + tid);
    if (rank == 0 && h % (s.heads / s.kv_heads) == 0 && tid < s.dim) {
        conv_keep(d, before, after, 1, s.off_q + kh * s.dim + tid);
        conv_keep(d, before, after, 1, s.off_k + kh * s.dim + tid);
    }
    if (h + 1 == s.heads && rank + 1 == ncta)   // padding up to the stride
        for (uint32_t i = s.heads * s.vdim + tid; i < d.ldo; i += 256) static_cast<float*>(d.out)[i] = 0.0f;
}

template <int E>
cudaError_t step_e(const DeltaStepArgs& a, cudaStream_t st, bool pdl) {
    const uint32_t ncta = a.d.s.vp / SCAN_COLS;
    cudaLaunchConfig_t lc = {};
    lc.gridDim = dim3(a.d.s.heads * ncta); lc.blockDim = dim3(256); lc.dynamicSmemBytes = (size_t)(a.a2.k + a.g2.k) * 4; lc.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = ncta; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    lc.attrs = at; lc.numAttrs = pdl ? 2 : 1;
    return cudaLaunchKernelEx(&lc, delta_step_kernel<E>, a);
}

template <int DP, int NW>
cudaError_t scan_inst(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    constexpr size_t smem = sizeof(ScanSmem<DP, NW>);
    const cudaError_t err = allow_smem(delta_scan_kernel<DP, NW>, smem, done);
    if (err != cudaSuccess) return err;
    return launch_pdl(delta_scan_kernel<DP, NW>, dim3(a.s.vp / (8 * NW), a.s.heads), dim3(NW * 32), smem, st, pdl, a, tokens);
}
template <int DP>
cudaError_t scan_dim(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    constexpr size_t smem = (size_t)3 * W * DP * sizeof(float);
    cudaError_t err = allow_smem(delta_pairs_kernel<DP>, smem, done);
    if (err != cudaSuccess) return err;
    err = launch_pdl(delta_pairs_kernel<DP>, dim3((tokens + W - 1) / W, a.s.heads), dim3(256), smem, st, pdl, a, tokens);
    if (err != cudaSuccess) return err;
    // few columns: narrower CTAs, so that more SMs have one
    return a.s.heads * (a.s.vp / 32) < 100 ? scan_inst<DP, 2>(a, tokens, st, pdl) : scan_inst<DP, 4>(a, tokens, st, pdl);
}

}  // namespace

template <int TAPS>
static cudaError_t prepare_taps(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const dim3 grid((tokens + 4 * PREP_TOKENS - 1) / (4 * PREP_TOKENS), a.s.kv_heads + a.s.heads);
    switch (a.s.dp) {
        case 64: return launch_pdl(delta_prepare_kernel<TAPS, 2>, grid, dim3(128), 0, st, pdl, a, tokens);
        case 128: return launch_pdl(delta_prepare_kernel<TAPS, 4>, grid, dim3(128), 0, st, pdl, a, tokens);
        case 256: return launch_pdl(delta_prepare_kernel<TAPS, 8>, grid, dim3(128), 0, st, pdl, a, tokens);
        default: return cudaErrorInvalidValue;
    }
}
cudaError_t launch_delta_prepare(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const cudaError_t err = a.s.taps == 4 ? prepare_taps<4>(a, tokens, st, pdl) : a.s.taps == 3 ? prepare_taps<3>(a, tokens, st, pdl)
                          : a.s.taps == 2 ? prepare_taps<2>(a, tokens, st, pdl) : prepare_taps<0>(a, tokens, st, pdl);
    if (err != cudaSuccess || a.s.taps <= 1) return err;
    return launch_pdl(conv_tail_kernel, dim3((a.s.conv_cols + 255) / 256), dim3(256), 0, st, pdl, a, tokens);
}

cudaError_t launch_delta_scan(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    switch (a.s.dp) {
        case 64: return scan_dim<64>(a, tokens, st, pdl);
        case 128: return scan_dim<128>(a, tokens, st, pdl);
        case 256: return scan_dim<256>(a, tokens, st, pdl);
        default: return cudaErrorInvalidValue;
    }
}

cudaError_t launch_delta_step(const DeltaStepArgs& a, cudaStream_t st, bool pdl) {
    if (!delta_step_fits(a)) return cudaErrorInvalidValue;
    switch (a.d.s.dp) {
        case 64: return step_e<8>(a, st, pdl);
        case 128: return step_e<16>(a, st, pdl);
        case 256: return step_e<32>(a, st, pdl);
        default: return cudaErrorInvalidValue;
    }
}

cudaError_t launch_delta_out(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const unsigned grid = (unsigned)(((size_t)tokens * a.s.heads + 7) / 8);
    return a.out_bf16 ? launch_pdl(delta_out_kernel<bf16>, dim3(grid), dim3(256), 0, st, pdl, a, tokens)
                      : launch_pdl(delta_out_kernel<float>, dim3(grid), dim3(256), 0, st, pdl, a, tokens);
}

}  // namespace alice
