// Delta rule with one decay per key channel. Per head, with a state S [dim][vdim] kept in f32:
//   S <- g * S (rows);  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
// A column of S never meets another one, so the recurrence runs column-parallel: eight lanes hold one column in registers
// for as long as the tokens last. Both products of a token are taken from the decayed column in one pass,
//   o = (gS)^T q + (k.q) u,   with k.q prepared per token,
// which leaves one eight-lane reduction on the token-to-token path.
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
    const float* w = a.conv_w + (size_t)c * taps;
    float v = 0.0f;
    for (int j = 0; j < taps; j++) {
        const int s = t - (taps - 1 - j);
        v = fmaf(w[j], s >= 0 ? a.y[(size_t)s * a.ldy + c] : before[(size_t)(taps - 1 + s) * a.s.conv_cols + c], v);
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

// One warp per (token, key head) or (token, value head).
__global__ void __launch_bounds__(256) delta_prepare_kernel(const __grid_constant__ DeltaArgs a, uint32_t tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const DeltaShape& s = a.s;
    const uint32_t lane = threadIdx.x & 31, per = s.kv_heads + s.heads;
    const size_t task = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (task >= (size_t)tokens * per) return;
    const float* before = conv_before(a);
    const uint32_t t = (uint32_t)(task / per), i = (uint32_t)(task % per);
    if (i < s.kv_heads) {
        constexpr int N = DELTA_MAX_DIM / 32;
        float q[N], k[N], sq = 0.0f, sk = 0.0f;
#pragma unroll
        for (int j = 0; j < N; j++) {
            const uint32_t d = lane + 32 * j;
            q[j] = k[j] = 0.0f;
            if (d < s.dim) {
                q[j] = conv_silu(a, before, (int)t, s.off_q + i * s.dim + d);
                k[j] = conv_silu(a, before, (int)t, s.off_k + i * s.dim + d);
            }
            sq = fmaf(q[j], q[j], sq); sk = fmaf(k[j], k[j], sk);
        }
        sq = warp_sum(sq); sk = warp_sum(sk);
        const float iq = __frcp_rn(__fsqrt_rn(sq + 1e-6f)) * __frcp_rn(__fsqrt_rn((float)s.dim)), ik = __frcp_rn(__fsqrt_rn(sk + 1e-6f));
        float dot = 0.0f;
        const size_t o = ((size_t)t * s.kv_heads + i) * s.dp;
#pragma unroll
        for (int j = 0; j < N; j++) {
            const uint32_t d = lane + 32 * j;
            q[j] *= iq; k[j] *= ik;
            dot = fmaf(q[j], k[j], dot);
            if (d < s.dp) { a.qn[o + d] = q[j]; a.kn[o + d] = k[j]; }
        }
        dot = warp_sum(dot);
        if (lane == 0) a.kq[(size_t)t * s.kv_heads + i] = dot;
    } else {
        const uint32_t h = i - s.kv_heads;
        const size_t o = ((size_t)t * s.heads + h) * s.vp;
        for (uint32_t d = lane; d < s.vp; d += 32) a.v[o + d] = d < s.vdim ? conv_silu(a, before, (int)t, s.off_v + h * s.vdim + d) : 0.0f;
        if (lane == 0) a.beta[(size_t)t * s.heads + h] = sigmoid_f(a.y[(size_t)t * a.ldy + s.off_b + h]);
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

constexpr int SCAN_COLS = 32, SCAN_CHUNK = 8;   // columns per CTA, tokens per staged chunk

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// E elements of a column per lane: element e of lane l is dim (e / 4) * 32 + l * 4 + e % 4.
template <int E>
struct ScanStage {
    float k[SCAN_CHUNK][8 * E], q[SCAN_CHUNK][8 * E], g[SCAN_CHUNK][8 * E], v[SCAN_CHUNK][SCAN_COLS];
    float beta[SCAN_CHUNK], kq[SCAN_CHUNK];
};

template <int E>
__device__ __forceinline__ void scan_fetch(ScanStage<E>& st, const DeltaArgs& a, uint32_t t0, uint32_t n, uint32_t h, uint32_t kh, uint32_t c0) {
    const DeltaShape& s = a.s;
    constexpr uint32_t P = 8 * E / 4;
    for (uint32_t i = threadIdx.x; i < n * P; i += 256) {
        const uint32_t j = i / P, d = i % P * 4;
        const size_t ko = ((size_t)(t0 + j) * s.kv_heads + kh) * s.dp + d;
        cp_async16(&st.k[j][d], a.kn + ko);
        cp_async16(&st.q[j][d], a.qn + ko);
        cp_async16(&st.g[j][d], a.g + ((size_t)(t0 + j) * s.heads + h) * s.dp + d);
    }
    for (uint32_t i = threadIdx.x; i < n * (SCAN_COLS / 4); i += 256) {
        const uint32_t j = i / (SCAN_COLS / 4), d = i % (SCAN_COLS / 4) * 4;
        cp_async16(&st.v[j][d], a.v + ((size_t)(t0 + j) * s.heads + h) * s.vp + c0 + d);
    }
    if (threadIdx.x < n) {
        st.beta[threadIdx.x] = a.beta[(size_t)(t0 + threadIdx.x) * s.heads + h];
        st.kq[threadIdx.x] = a.kq[(size_t)(t0 + threadIdx.x) * s.kv_heads + kh];
    }
}

template <int E>
__global__ void __launch_bounds__(256) delta_scan_kernel(const __grid_constant__ DeltaArgs a, uint32_t tokens) {
    extern __shared__ __align__(16) uint8_t smem[];
    auto* stage = reinterpret_cast<ScanStage<E>*>(smem);   // two
    __shared__ float os[SCAN_CHUNK][SCAN_COLS];
    const DeltaShape& s = a.s;
    const uint32_t h = blockIdx.y, kh = h / (s.heads / s.kv_heads), c0 = blockIdx.x * SCAN_COLS;
    const uint32_t lane = threadIdx.x & 31, l = lane & 7, col = (threadIdx.x >> 5) * 4 + (lane >> 3);
    float* sp = a.state + ((size_t)h * s.vp + c0 + col) * s.dp + l * 4;
    pdl_launch_dependents();
    pdl_wait();
    float S[E];
#pragma unroll
    for (int e = 0; e < E; e += 4) {
        const float4 f = *reinterpret_cast<const float4*>(sp + e * 8);
        S[e] = f.x; S[e + 1] = f.y; S[e + 2] = f.z; S[e + 3] = f.w;
    }
    scan_fetch<E>(stage[0], a, 0, min(tokens, (uint32_t)SCAN_CHUNK), h, kh, c0);
    cp_commit();
    for (uint32_t t0 = 0, b = 0; t0 < tokens; t0 += SCAN_CHUNK, b ^= 1) {
        const uint32_t n = min(tokens - t0, (uint32_t)SCAN_CHUNK);
        if (t0 + SCAN_CHUNK < tokens) scan_fetch<E>(stage[b ^ 1], a, t0 + SCAN_CHUNK, min(tokens - t0 - SCAN_CHUNK, (uint32_t)SCAN_CHUNK), h, kh, c0);
        cp_commit();
        cp_wait<1>();
        __syncthreads();
        const ScanStage<E>& st = stage[b];
        for (uint32_t j = 0; j < n; j++) {
            float k[E], dk = 0.0f, dq = 0.0f, dk2 = 0.0f, dq2 = 0.0f;
#pragma unroll
            for (int e = 0; e < E; e += 4) {
                const float4 kk = *reinterpret_cast<const float4*>(&st.k[j][e * 8 + l * 4]), qq = *reinterpret_cast<const float4*>(&st.q[j][e * 8 + l * 4]),
                             gg = *reinterpret_cast<const float4*>(&st.g[j][e * 8 + l * 4]);
                S[e] *= gg.x; S[e + 1] *= gg.y; S[e + 2] *= gg.z; S[e + 3] *= gg.w;
                dk = fmaf(S[e], kk.x, dk); dk2 = fmaf(S[e + 1], kk.y, dk2); dk = fmaf(S[e + 2], kk.z, dk); dk2 = fmaf(S[e + 3], kk.w, dk2);
                dq = fmaf(S[e], qq.x, dq); dq2 = fmaf(S[e + 1], qq.y, dq2); dq = fmaf(S[e + 2], qq.z, dq); dq2 = fmaf(S[e + 3], qq.w, dq2);
                k[e] = kk.x; k[e + 1] = kk.y; k[e + 2] = kk.z; k[e + 3] = kk.w;
            }
            dk += dk2; dq += dq2;
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) {
                dk += __shfl_xor_sync(0xffffffffu, dk, o);
                dq += __shfl_xor_sync(0xffffffffu, dq, o);
            }
            const float u = st.beta[j] * (st.v[j][col] - dk);
#pragma unroll
            for (int e = 0; e < E; e++) S[e] = fmaf(k[e], u, S[e]);
            if (l == 0) os[j][col] = fmaf(st.kq[j], u, dq);
        }
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < n * SCAN_COLS; i += 256) {
            const uint32_t j = i / SCAN_COLS, c = i % SCAN_COLS;
            if (c0 + c < s.vdim) a.o[((size_t)(t0 + j) * s.heads + h) * s.vdim + c0 + c] = os[j][c];
        }
        __syncthreads();
    }
#pragma unroll
    for (int e = 0; e < E; e += 4) *reinterpret_cast<float4*>(sp + e * 8) = make_float4(S[e], S[e + 1], S[e + 2], S[e + 3]);
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

template <int E>
cudaError_t scan_e(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    constexpr size_t smem = 2 * sizeof(ScanStage<E>);
    const cudaError_t err = allow_smem(delta_scan_kernel<E>, smem, done);
    if (err != cudaSuccess) return err;
    return launch_pdl(delta_scan_kernel<E>, dim3(a.s.vp / SCAN_COLS, a.s.heads), dim3(256), smem, st, pdl, a, tokens);
}

}  // namespace

cudaError_t launch_delta_prepare(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const size_t tasks = (size_t)tokens * (a.s.kv_heads + a.s.heads);
    cudaError_t err = launch_pdl(delta_prepare_kernel, dim3((unsigned)((tasks + 7) / 8)), dim3(256), 0, st, pdl, a, tokens);
    if (err != cudaSuccess || a.s.taps <= 1) return err;
    return launch_pdl(conv_tail_kernel, dim3((a.s.conv_cols + 255) / 256), dim3(256), 0, st, pdl, a, tokens);
}

cudaError_t launch_delta_scan(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    switch (a.s.dp) {
        case 32: return scan_e<4>(a, tokens, st, pdl);
        case 64: return scan_e<8>(a, tokens, st, pdl);
        case 128: return scan_e<16>(a, tokens, st, pdl);
        case 256: return scan_e<32>(a, tokens, st, pdl);
        default: return cudaErrorInvalidValue;
    }
}

cudaError_t launch_delta_step(const DeltaStepArgs& a, cudaStream_t st, bool pdl) {
    if (!delta_step_fits(a.d.s) || (size_t)(a.a2.k + a.g2.k) * 4 > 32 * 1024) return cudaErrorInvalidValue;
    switch (a.d.s.dp) {
        case 32: return step_e<4>(a, st, pdl);
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
