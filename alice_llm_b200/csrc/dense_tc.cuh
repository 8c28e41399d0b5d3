// bf16 tiled product on the fifth-generation tensor cores: C[t][n] = sum_k A[t][k] W[n][k].
//
// Persistent, one CTA per SM, six warps: warp 0 copies 128 x 64 and BN x 64 tiles by TMA (128-byte swizzle) into a ring of
// stages, warp 1 issues tcgen05.mma from one thread into one of two TMEM accumulators, warps 2-5 drain the other one and
// apply the epilogue. Every wait is bounded: when one runs out the kernel records it in the status word, lets its copies and
// products finish, gives its TMEM back and returns.
#pragma once
#include "dense_epi.cuh"
#include "tc_dev.cuh"

namespace alice {

constexpr int TC_BM = 128, TC_BK = 64, TC_THREADS = 192;
template <int BN>
struct TcGeom {
    static constexpr int STAGES = BN == 256 ? 4 : 6;
    static constexpr uint32_t A_BYTES = TC_BM * TC_BK * 2, B_BYTES = BN * TC_BK * 2, STAGE = A_BYTES + B_BYTES;
    static constexpr size_t SMEM = (size_t)STAGES * STAGE + 1024;   // + alignment of the ring
    static constexpr uint32_t TMEM_COLS = 2 * BN;
};
constexpr int KERR_TC_WAIT = 7;   // a wait inside the tensor-core product

struct TcArgs {
    GemmOp op;
    CUtensorMap ta, tw;
    int* status;
};

// 32 consecutive columns of one token.
template <int EPI>
__device__ __forceinline__ void epi_32(const GemmOp& op, uint32_t t, uint32_t n, const float (&v)[32]) {
    const size_t o = (size_t)t * op.ldo + n;
    const bool whole = n + 32 <= op.w.n && (o & 7) == 0;
    if constexpr (EPI == EPI_STORE) {
        if (whole && !op.out_bf16) {
            float4* p = reinterpret_cast<float4*>(static_cast<float*>(op.out) + o);
#pragma unroll
            for (int i = 0; i < 8; i++) p[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
            if (!op.out2 || n + 32 <= op.col2) return;
#pragma unroll
            for (int i = 0; i < 32; i++)
                if (n + i >= op.col2) put(op.out2 + (size_t)t * op.ld2 + (n + i - op.col2), v[i]);
            return;
        }
        if (whole) {
            uint4* p = reinterpret_cast<uint4*>(static_cast<bf16*>(op.out) + o);
#pragma unroll
            for (int i = 0; i < 4; i++) {
                uint32_t w[4];
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const __nv_bfloat162 b = __floats2bfloat162_rn(v[8 * i + 2 * j], v[8 * i + 2 * j + 1]);
                    w[j] = *reinterpret_cast<const uint32_t*>(&b);
                }
                p[i] = make_uint4(w[0], w[1], w[2], w[3]);
            }
            if (!op.out2) return;
#pragma unroll
            for (int i = 0; i < 32; i++)
                if (n + i >= op.col2) put(op.out2 + (size_t)t * op.ld2 + (n + i - op.col2), v[i]);
            return;
        }
    } else if constexpr (EPI == EPI_RESID) {
        if (whole) {
            float4* p = reinterpret_cast<float4*>(static_cast<float*>(op.out) + o);
#pragma unroll
            for (int i = 0; i < 8; i++) {
                float4 x = p[i];
                const float4 s = op.scale ? __ldg(reinterpret_cast<const float4*>(op.scale + n) + i) : make_float4(1.f, 1.f, 1.f, 1.f);
                const float4 b = op.bias ? __ldg(reinterpret_cast<const float4*>(op.bias + n) + i) : make_float4(0.f, 0.f, 0.f, 0.f);
                x.x = op.alpha * x.x + s.x * (v[4 * i] + b.x); x.y = op.alpha * x.y + s.y * (v[4 * i + 1] + b.y);
                x.z = op.alpha * x.z + s.z * (v[4 * i + 2] + b.z); x.w = op.alpha * x.w + s.w * (v[4 * i + 3] + b.w);
                p[i] = x;
            }
            return;
        }
    } else {
        if (whole) {
            float4* p = reinterpret_cast<float4*>(static_cast<float*>(op.out) + o);
            const uint32_t head = EPI == EPI_DECAY ? n / op.dim : 0;
            const bool one = EPI == EPI_DECAY && (n + 31) / op.dim == head;   // one head in these columns: one rate
            const float rate = one ? expf(__ldg(op.a_log + head)) : 0.0f;
#pragma unroll
            for (int i = 0; i < 8; i++) {
                float r[4];
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const uint32_t c = n + 4 * i + j;
                    if constexpr (EPI == EPI_DECAY) r[j] = expf(-(one ? rate : expf(__ldg(op.a_log + c / op.dim))) * softplus_f(v[4 * i + j] + __ldg(op.bias + c)));
                    else r[j] = sigmoid_f(v[4 * i + j]);
                }
                p[i] = make_float4(r[0], r[1], r[2], r[3]);
            }
            return;
        }
    }
#pragma unroll
    for (int i = 0; i < 32; i++)
        if (n + i < op.w.n) epi_one<EPI>(op, t, n + i, v[i]);
}

__device__ __forceinline__ void epi_swiglu_32(const GemmOp& op, uint32_t t, uint32_t c, const float (&g)[32], const float (&u)[32]) {
    const size_t o = (size_t)t * op.ldo + c;
#pragma unroll
    for (int i = 0; i < 4; i++) {
        float r[8];
#pragma unroll
        for (int j = 0; j < 8; j++) {
            const int k = 8 * i + j;
            r[j] = op.bias ? silu_ref(g[k] + __ldg(op.bias + c + k)) * (u[k] + __ldg(op.bias2 + c + k)) : silu_ref(g[k]) * u[k];
        }
        uint32_t w[4];
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(r[2 * j], r[2 * j + 1]);
            w[j] = *reinterpret_cast<const uint32_t*>(&b);
        }
        reinterpret_cast<uint4*>(static_cast<bf16*>(op.out) + o)[i] = make_uint4(w[0], w[1], w[2], w[3]);
    }
}

template <int BN, int EPI>
__global__ void __launch_bounds__(TC_THREADS, 1) gemm_tc_kernel(const __grid_constant__ TcArgs a) {
    using G = TcGeom<BN>;
    extern __shared__ uint8_t raw[];
    __shared__ __align__(8) uint64_t full_[G::STAGES], empty_[G::STAGES], tfull_[2], tempty_[2], drain_;
    __shared__ uint32_t tmem_base;
    const uint32_t ring = (smem_u32(raw) + 1023u) & ~1023u;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const GemmOp& op = a.op;
    auto bar = [](uint64_t* b, int i) { return smem_u32(b + i); };
    pdl_launch_dependents();
    if (threadIdx.x == 0) {
        for (int i = 0; i < G::STAGES; i++) { mbar_init(bar(full_, i), 1); mbar_init(bar(empty_, i), 1); }
        for (int i = 0; i < 2; i++) { mbar_init(bar(tfull_, i), 1); mbar_init(bar(tempty_, i), 128); }
        mbar_init(smem_u32(&drain_), 1);
        mbar_fence_init();
        fence_proxy_async();
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base)), "n"(G::TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_base;
    pdl_wait();

    const uint32_t tiles_t = (op.tokens + TC_BM - 1) / TC_BM, tiles_n = (op.w.n + BN - 1) / BN, tiles = tiles_t * tiles_n;
    const uint32_t ksteps = op.w.k / TC_BK;
    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x) {
                const int t0 = (int)(tile % tiles_t * TC_BM), n0 = (int)(tile / tiles_t * BN);
                for (uint32_t k = 0; k < ksteps; k++, it++) {
                    const int s = (int)(it % G::STAGES);
                    if (!mbar_wait(bar(empty_, s), ((it / G::STAGES) & 1) ^ 1)) { atomicCAS(a.status, 0, KERR_TC_WAIT); ok = false; break; }
                    const uint32_t dst = ring + s * G::STAGE;
                    mbar_arrive_expect_tx(bar(full_, s), G::STAGE);
                    tma_2d(dst, &a.ta, (int)(k * TC_BK), t0, bar(full_, s));
                    tma_2d(dst + G::A_BYTES, &a.tw, (int)(k * TC_BK), n0, bar(full_, s));
                }
            }
            // every copy has landed before the CTA may leave
            const uint32_t last = it < (uint32_t)G::STAGES ? it : (uint32_t)G::STAGES;
            for (uint32_t j = it - last; j < it; j++) mbar_wait(bar(full_, (int)(j % G::STAGES)), (j / G::STAGES) & 1);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = mma_desc(TC_BM, BN);
            uint32_t it = 0, i = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, i++) {
                const int b = (int)(i & 1);
                if (!mbar_wait(bar(tempty_, b), ((i >> 1) & 1) ^ 1)) { atomicCAS(a.status, 0, KERR_TC_WAIT); break; }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t d = tmem + (uint32_t)b * BN;
                for (uint32_t k = 0; k < ksteps; k++, it++) {
                    const int s = (int)(it % G::STAGES);
                    if (!mbar_wait(bar(full_, s), (it / G::STAGES) & 1)) { atomicCAS(a.status, 0, KERR_TC_WAIT); ok = false; break; }
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint64_t da = smem_desc(ring + s * G::STAGE), db = smem_desc(ring + s * G::STAGE + G::A_BYTES);
#pragma unroll
                    for (int kk = 0; kk < TC_BK / 16; kk++) mma_f16(d, da + 2 * kk, db + 2 * kk, idesc, k > 0 || kk > 0);
                    mma_commit(bar(empty_, s));
                }
                if (ok) mma_commit(bar(tfull_, b));
            }
            mma_commit(smem_u32(&drain_));
            if (!mbar_wait(smem_u32(&drain_), 0)) atomicCAS(a.status, 0, KERR_TC_WAIT);
        }
    } else {
        const uint32_t quad = warp & 3, row = quad * 32 + lane;
        uint32_t i = 0;
        for (uint32_t tile = blockIdx.x; tile < tiles; tile += gridDim.x, i++) {
            const int b = (int)(i & 1);
            const uint32_t t = tile % tiles_t * TC_BM + row, n0 = tile / tiles_t * BN;
            const bool ok = mbar_wait(bar(tfull_, b), (i >> 1) & 1);
            if (!__all_sync(0xffffffffu, ok)) { if (lane == 0) atomicCAS(a.status, 0, KERR_TC_WAIT); break; }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t base = tmem + (uint32_t)b * BN + ((quad * 32) << 16);
            if constexpr (EPI == EPI_SWIGLU) {
#pragma unroll 1
                for (uint32_t c = 0; c < BN; c += 128) {
                    if (n0 + c >= op.w.n) break;
#pragma unroll 1
                    for (uint32_t j = 0; j < 64; j += 32) {
                        float g[32], u[32];
                        tmem_ld32(g, base + c + j);
                        tmem_ld32(u, base + c + 64 + j);
                        if (t < op.tokens) epi_swiglu_32(op, t, (n0 + c) / 2 + j, g, u);
                    }
                }
            } else {
#pragma unroll 1
                for (uint32_t c = 0; c < BN; c += 32) {
                    if (n0 + c >= op.w.n) break;
                    float v[32];
                    tmem_ld32(v, base + c);
                    if (t < op.tokens) epi_32<EPI>(op, t, n0 + c, v);
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(bar(tempty_, b));
        }
    }
    __syncwarp();
    __syncthreads();
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(G::TMEM_COLS));
}

}  // namespace alice
