// Many tokens against dense bfloat16 rows. f32 inputs: register-tiled f32 arithmetic (every product and sum in 32 bits).
#include "dense_epi.cuh"

namespace alice {
namespace {

constexpr int BM = 64, BN = 128, BK = 16;

__device__ __forceinline__ void load_a4(float (&r)[4], const float* p) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    r[0] = v.x; r[1] = v.y; r[2] = v.z; r[3] = v.w;
}
__device__ __forceinline__ void load_a4(float (&r)[4], const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = bf2(v.x), b = bf2(v.y);
    r[0] = a.x; r[1] = a.y; r[2] = b.x; r[3] = b.y;
}

// 256 threads; a thread owns 4 tokens x (4 columns of the tile's first half + the same 4 of its second half).
template <class AT, int EPI>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const __grid_constant__ GemmOp op) {
    __shared__ __align__(16) float As[BK][BM + 4], Bs[BK][BN + 4];
    const uint32_t tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const uint32_t t0 = blockIdx.y * BM, n0 = blockIdx.x * BN, k_end = op.w.k;
    const uint32_t ar = tid >> 2, ak = (tid & 3) * 4, br = tid >> 1, bk = (tid & 1) * 8;
    pdl_launch_dependents();
    pdl_wait();
    const AT* ap = static_cast<const AT*>(op.a) + (size_t)(t0 + ar) * op.lda + ak;
    const bf16* bp = op.w.w + (size_t)(n0 + br) * op.w.k + bk;
    const bool a_ok = t0 + ar < op.tokens, b_ok = n0 + br < op.w.n;
    float acc[4][8] = {};
    float ra[4] = {};
    uint4 rb = make_uint4(0, 0, 0, 0);
    if (a_ok) load_a4(ra, ap);
    if (b_ok) rb = __ldg(reinterpret_cast<const uint4*>(bp));
    for (uint32_t k = 0; k < k_end; k += BK) {
#pragma unroll
        for (int i = 0; i < 4; i++) As[ak + i][ar] = ra[i];
        const float2 b0 = bf2(rb.x), b1 = bf2(rb.y), b2 = bf2(rb.z), b3 = bf2(rb.w);
        Bs[bk + 0][br] = b0.x; Bs[bk + 1][br] = b0.y; Bs[bk + 2][br] = b1.x; Bs[bk + 3][br] = b1.y;
        Bs[bk + 4][br] = b2.x; Bs[bk + 5][br] = b2.y; Bs[bk + 6][br] = b3.x; Bs[bk + 7][br] = b3.y;
        __syncthreads();
        if (k + BK < k_end) {
            if (a_ok) load_a4(ra, ap + k + BK);
            if (b_ok) rb = __ldg(reinterpret_cast<const uint4*>(bp + k + BK));
        }
#pragma unroll
        for (int kk = 0; kk < BK; kk++) {
            const float4 a = *reinterpret_cast<const float4*>(&As[kk][ty * 4]);
            const float4 b = *reinterpret_cast<const float4*>(&Bs[kk][tx * 4]), c = *reinterpret_cast<const float4*>(&Bs[kk][64 + tx * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[8] = {b.x, b.y, b.z, b.w, c.x, c.y, c.z, c.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 8; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t t = t0 + ty * 4 + i;
        if (t >= op.tokens) break;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            if constexpr (EPI == EPI_SWIGLU) {
                epi_swiglu(op, t, n0 / 2 + tx * 4 + j, acc[i][j], acc[i][4 + j]);
            } else {
                if (n0 + tx * 4 + j < op.w.n) epi_one<EPI>(op, t, n0 + tx * 4 + j, acc[i][j]);
                if (n0 + 64 + tx * 4 + j < op.w.n) epi_one<EPI>(op, t, n0 + 64 + tx * 4 + j, acc[i][4 + j]);
            }
        }
    }
}

template <class AT>
cudaError_t launch_f32(const GemmOp& op, cudaStream_t st, bool pdl) {
    const dim3 grid((op.w.n + BN - 1) / BN, (op.tokens + BM - 1) / BM);
    switch (op.epi) {
        case EPI_STORE: return launch_pdl(gemm_f32_kernel<AT, EPI_STORE>, grid, dim3(256), 0, st, pdl, op);
        case EPI_SWIGLU: return launch_pdl(gemm_f32_kernel<AT, EPI_SWIGLU>, grid, dim3(256), 0, st, pdl, op);
        case EPI_RESID: return launch_pdl(gemm_f32_kernel<AT, EPI_RESID>, grid, dim3(256), 0, st, pdl, op);
        case EPI_DECAY: return launch_pdl(gemm_f32_kernel<AT, EPI_DECAY>, grid, dim3(256), 0, st, pdl, op);
        case EPI_SIGMOID: return launch_pdl(gemm_f32_kernel<AT, EPI_SIGMOID>, grid, dim3(256), 0, st, pdl, op);
        default: return cudaErrorInvalidValue;
    }
}

}  // namespace

cudaError_t launch_dense_gemm(const GemmOp& op, int* status, cudaStream_t st, bool pdl) {
    (void)status;
    if (!op.tokens || !op.w.n || op.w.k % DENSE_PAD || op.lda % 8 || ((uintptr_t)op.a & 15) || (op.epi == EPI_SWIGLU && op.w.n % 128)) return cudaErrorInvalidValue;
    return op.a_bf16 ? launch_f32<bf16>(op, st, pdl) : launch_f32<float>(op, st, pdl);
}

}  // namespace alice
