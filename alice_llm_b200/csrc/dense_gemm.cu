// Many tokens against dense bfloat16 rows. f32 inputs: register-tiled f32 arithmetic (every product and sum in 32 bits).
// bf16 inputs: tensor cores (dense_tc.cuh).
#include "dense_tc.cuh"

namespace alice {
namespace {

constexpr int BM = 64, BN = 128, BK = 16;

__device__ __forceinline__ void load_a4(float (&r)[4], const float* p) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    r[0] = v.x; r[1] = v.y; r[2] = v.z; r[3] = v.w;
}

// 256 threads; a thread owns 4 tokens x (4 columns of the tile's first half + the same 4 of its second half).
template <int EPI>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const __grid_constant__ GemmOp op) {
    __shared__ __align__(16) float As[BK][BM + 4], Bs[BK][BN + 4];
    const uint32_t tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const uint32_t t0 = blockIdx.y * BM, n0 = blockIdx.x * BN, k_end = op.w.k;
    const uint32_t ar = tid >> 2, ak = (tid & 3) * 4, br = tid >> 1, bk = (tid & 1) * 8;
    pdl_launch_dependents();
    pdl_wait();
    const float* ap = static_cast<const float*>(op.a) + (size_t)(t0 + ar) * op.lda + ak;
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

cudaError_t launch_f32(const GemmOp& op, cudaStream_t st, bool pdl) {
    const dim3 grid((op.w.n + BN - 1) / BN, (op.tokens + BM - 1) / BM);
    switch (op.epi) {
        case EPI_STORE: return launch_pdl(gemm_f32_kernel<EPI_STORE>, grid, dim3(256), 0, st, pdl, op);
        case EPI_SWIGLU: return launch_pdl(gemm_f32_kernel<EPI_SWIGLU>, grid, dim3(256), 0, st, pdl, op);
        case EPI_RESID: return launch_pdl(gemm_f32_kernel<EPI_RESID>, grid, dim3(256), 0, st, pdl, op);
        case EPI_DECAY: return launch_pdl(gemm_f32_kernel<EPI_DECAY>, grid, dim3(256), 0, st, pdl, op);
        case EPI_SIGMOID: return launch_pdl(gemm_f32_kernel<EPI_SIGMOID>, grid, dim3(256), 0, st, pdl, op);
        default: return cudaErrorInvalidValue;
    }
}

template <int BN, int EPI>
cudaError_t tc_inst(const TcArgs& a, uint32_t grid, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    const cudaError_t err = allow_smem(gemm_tc_kernel<BN, EPI>, TcGeom<BN>::SMEM, done);
    if (err != cudaSuccess) return err;
    return launch_pdl(gemm_tc_kernel<BN, EPI>, dim3(grid), dim3(TC_THREADS), TcGeom<BN>::SMEM, st, pdl, a);
}
template <int BN>
cudaError_t tc_epi(const TcArgs& a, uint32_t grid, cudaStream_t st, bool pdl) {
    switch (a.op.epi) {
        case EPI_STORE: return tc_inst<BN, EPI_STORE>(a, grid, st, pdl);
        case EPI_SWIGLU: return tc_inst<BN, EPI_SWIGLU>(a, grid, st, pdl);
        case EPI_RESID: return tc_inst<BN, EPI_RESID>(a, grid, st, pdl);
        case EPI_DECAY: return tc_inst<BN, EPI_DECAY>(a, grid, st, pdl);
        case EPI_SIGMOID: return tc_inst<BN, EPI_SIGMOID>(a, grid, st, pdl);
        default: return cudaErrorInvalidValue;
    }
}

cudaError_t launch_tc(const GemmOp& op, int num_sms, int* status, cudaStream_t st, bool pdl) {
    if (!encode_fn()) return cudaErrorNotSupported;
    TcArgs a;
    a.op = op; a.status = status;
    const uint32_t tt = (op.tokens + TC_BM - 1) / TC_BM;
    // wide tiles when they still give every SM one
    const bool wide = tt * ((op.w.n + 255) / 256) >= (uint32_t)num_sms;
    const uint32_t bn = wide ? 256 : 128, tiles = tt * ((op.w.n + bn - 1) / bn);
    if (!tile_map(&a.ta, op.a, op.tokens, op.w.k, op.lda, TC_BM) || !tile_map(&a.tw, op.w.w, op.w.n, op.w.k, op.w.k, bn)) return cudaErrorInvalidValue;
    const uint32_t grid = std::min(tiles, (uint32_t)num_sms);
    return wide ? tc_epi<256>(a, grid, st, pdl) : tc_epi<128>(a, grid, st, pdl);
}

}  // namespace

cudaError_t launch_dense_gemm(const GemmOp& op, int num_sms, int* status, cudaStream_t st, bool pdl) {
    if (!op.tokens || !op.w.n || op.w.k % DENSE_PAD || op.lda % 8 || ((uintptr_t)op.a & 15) || ((uintptr_t)op.out & 15) || (op.epi == EPI_SWIGLU && op.w.n % 128))
        return cudaErrorInvalidValue;
    if (!op.a_bf16) return launch_f32(op, st, pdl);
    if (op.epi == EPI_SWIGLU && (!op.out_bf16 || op.ldo % 8)) return cudaErrorInvalidValue;
    return launch_tc(op, num_sms, status, st, pdl);
}

}  // namespace alice
