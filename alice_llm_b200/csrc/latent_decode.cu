// Attention of single tokens over a bfloat16 latent cache on the tensor cores. The cached row is shared by all heads, so
// sixteen heads are the rows of one product: scores = Q [16 x (cp + rp)] K^T, sums = P [16 x keys] C. Queries and softmax
// weights enter as bf16 pairs (value and remainder); everything between is f32.
#include "dense_dev.cuh"
#include "mixers.cuh"
#include "mma_sync.cuh"

namespace alice {
namespace {

constexpr uint32_t LD_KEYS = 32, LD_HEADS = 16, LD_STAGES = 2;   // a deeper ring measured no faster

// grid (head groups of 16, splits, tokens), 8 warps. NT: 8-column tiles of the weighted sum per warp (8 * NT * 8 >= cp).
template <int NT>
__global__ void __launch_bounds__(256, 1) latent_decode_kernel(const __grid_constant__ LatentArgs a) {
    extern __shared__ __align__(128) uint8_t sm[];
    __shared__ float sc[2][LD_HEADS][LD_KEYS + 4], mrow[LD_HEADS], lrow[LD_HEADS], frow[LD_HEADS];
    __shared__ __align__(16) bf16 ph[LD_HEADS][LD_KEYS + 8], pl[LD_HEADS][LD_KEYS + 8];
    const LatentShape& s = a.s;
    const uint32_t width = s.cp + s.rp, ld = width + 8;   // row stride: eight rows in different banks (width is a multiple of 16)
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, t = blockIdx.z, h0 = blockIdx.x * LD_HEADS;
    auto* qh = reinterpret_cast<bf16*>(sm);
    bf16* ql = qh + LD_HEADS * ld;
    bf16* kt = ql + LD_HEADS * ld;                        // LD_STAGES tiles of [LD_KEYS][ld]
    const uint32_t qh_s = smem_u32(qh), ql_s = smem_u32(ql), kt_s = smem_u32(kt), tile_bytes = LD_KEYS * ld * 2;
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t ctx = (uint32_t)*a.pos + t + 1;
    const uint32_t share = ((ctx + gridDim.y - 1) / gridDim.y + LD_KEYS - 1) / LD_KEYS * LD_KEYS;
    const uint32_t lo = min(ctx, blockIdx.y * share), hi = min(ctx, lo + share);
    float* out = a.part + ((size_t)t * gridDim.y + blockIdx.y) * s.heads * (s.cp + 2);
    if (lo >= hi) {   // nothing here: the join gives this share weight zero
        if (tid < LD_HEADS && h0 + tid < s.heads) { out[(size_t)(h0 + tid) * (s.cp + 2) + s.cp] = -INFINITY; out[(size_t)(h0 + tid) * (s.cp + 2) + s.cp + 1] = 0.0f; }
        return;
    }
    const bf16* cache = static_cast<const bf16*>(a.cache);
    auto fetch = [&](uint32_t k0, uint32_t b) {
        const uint32_t row = tid / 8, j = min(k0 + row, hi - 1);   // eight threads a row
        const bf16* src = cache + (size_t)j * width;
        const uint32_t dst = kt_s + b * tile_bytes + row * ld * 2;
        if (k0 < hi)
            for (uint32_t c = tid % 8 * 8; c < width; c += 64) cp16(dst + c * 2, src + c, k0 + row < hi);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (uint32_t i = 0; i + 1 < LD_STAGES; i++) fetch(lo + i * LD_KEYS, i);
    static_assert(LD_KEYS * 8 == 256, "a tile is fetched in one round of rows");
#pragma unroll
    for (uint32_t r = warp; r < LD_HEADS; r += 8) {
        const float* q = a.ql + ((size_t)t * s.heads + min(h0 + r, s.heads - 1)) * width;
        const float f = h0 + r < s.heads ? s.scale : 0.0f;
#pragma unroll 5
        for (uint32_t c = lane * 4; c < width; c += 128) {
            const float4 v = *reinterpret_cast<const float4*>(q + c);
            const float x0 = v.x * f, x1 = v.y * f, x2 = v.z * f, x3 = v.w * f;
            const uint2 hw = make_uint2(pack_bf16(x0, x1), pack_bf16(x2, x3));
            const float2 h01 = bf2(hw.x), h23 = bf2(hw.y);
            *reinterpret_cast<uint2*>(qh + r * ld + c) = hw;
            *reinterpret_cast<uint2*>(ql + r * ld + c) = make_uint2(pack_bf16(x0 - h01.x, x1 - h01.y), pack_bf16(x2 - h23.x, x3 - h23.y));
        }
    }
    if (tid < LD_HEADS) { mrow[tid] = -INFINITY; lrow[tid] = 0.0f; }
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const uint32_t c0 = warp * NT * 8;                    // this warp's latent columns

    for (uint32_t k0 = lo, b = 0; k0 < hi; k0 += LD_KEYS, b = (b + 1) % LD_STAGES) {
        fetch(k0 + (LD_STAGES - 1) * LD_KEYS, (b + LD_STAGES - 1) % LD_STAGES);   // into the tile that was read last
        asm volatile("cp.async.wait_group %0;" ::"n"(LD_STAGES - 1) : "memory");
        __syncthreads();
        const uint32_t kb = kt_s + b * tile_bytes;
        {   // scores: four warps of eight keys over the first half of the columns, four over the second
            float d[4][4] = {};
            const uint32_t nt = warp & 3, mid = width / 64 * 32, stop = warp < 4 ? mid : width;
            const uint32_t qa = ((lane % 16) * ld + lane / 16 * 8) * 2, ka = kb + ((nt * 8 + lane % 8) * ld + lane / 8 * 8) * 2;
            uint32_t kk = warp < 4 ? 0 : mid;
#pragma unroll 3
            for (; kk + 32 <= stop; kk += 32) {   // two k-steps of the key operand per load
                uint32_t k4[4], q4[4];
                ldsm4(k4, ka + kk * 2);
                ldsm4(q4, qh_s + qa + kk * 2); mma16816(d[0], q4, k4[0], k4[1]);
                ldsm4(q4, ql_s + qa + kk * 2); mma16816(d[1], q4, k4[0], k4[1]);
                ldsm4(q4, qh_s + qa + kk * 2 + 32); mma16816(d[2], q4, k4[2], k4[3]);
                ldsm4(q4, ql_s + qa + kk * 2 + 32); mma16816(d[3], q4, k4[2], k4[3]);
            }
            if (kk < stop) {   // an odd k-step: its second half would lie past the row
                uint32_t k2[2], q4[4];
                ldsm2(k2, kb + ((nt * 8 + lane % 8) * ld + (lane / 8 & 1) * 8) * 2 + kk * 2);
                ldsm4(q4, qh_s + qa + kk * 2); mma16816(d[0], q4, k2[0], k2[1]);
                ldsm4(q4, ql_s + qa + kk * 2); mma16816(d[1], q4, k2[0], k2[1]);
            }
            const uint32_t r = lane / 4, c = nt * 8 + (lane & 3) * 2;
            float (&out_sc)[LD_HEADS][LD_KEYS + 4] = sc[warp >> 2];
            out_sc[r][c] = (d[0][0] + d[2][0]) + (d[1][0] + d[3][0]); out_sc[r][c + 1] = (d[0][1] + d[2][1]) + (d[1][1] + d[3][1]);
            out_sc[r + 8][c] = (d[0][2] + d[2][2]) + (d[1][2] + d[3][2]); out_sc[r + 8][c + 1] = (d[0][3] + d[2][3]) + (d[1][3] + d[3][3]);
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; i++) {   // softmax of two heads per warp, a key per lane
            const uint32_t r = warp * 2 + i;
            float x = k0 + lane < hi ? sc[0][r][lane] + sc[1][r][lane] : -INFINITY;
            const float m0 = mrow[r], top = fmaxf(m0, warp_max(x)), f = expf(m0 - top);
            x = expf(x - top);
            const float sum = warp_sum(x);
            const bf16 xb = __float2bfloat16_rn(x);
            ph[r][lane] = xb;
            pl[r][lane] = __float2bfloat16_rn(x - __bfloat162float(xb));
            __syncwarp();
            if (lane == 0) { mrow[r] = top; lrow[r] = fmaf(lrow[r], f, sum); frow[r] = f; }
        }
        __syncthreads();
        const float f0 = frow[lane / 4], f1 = frow[lane / 4 + 8];
#pragma unroll
        for (int i = 0; i < NT; i++) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
        const uint32_t pa = ((lane % 16) * (LD_KEYS + 8) + lane / 16 * 8) * 2;
#pragma unroll
        for (uint32_t kk = 0; kk < LD_KEYS; kk += 16) {
            uint32_t p4[4], r4[4];
            ldsm4(p4, smem_u32(ph) + pa + kk * 2);
            ldsm4(r4, smem_u32(pl) + pa + kk * 2);
#pragma unroll
            for (int i = 0; i < NT; i += 2) {
                if (c0 + i * 8 >= s.cp) break;            // cp is a multiple of 64: whole pairs of tiles
                uint32_t v4[4];
                ldsm4t(v4, kb + ((kk + lane % 16) * ld + c0 + i * 8 + lane / 16 * 8) * 2);
                mma16816(o[i], p4, v4[0], v4[1]);
                mma16816(o[i + 1], p4, v4[2], v4[3]);
                mma16816(o[i], r4, v4[0], v4[1]);
                mma16816(o[i + 1], r4, v4[2], v4[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NT; i++) {
        const uint32_t c = c0 + i * 8 + (lane & 3) * 2;
        if (c >= s.cp) break;
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const uint32_t h = h0 + lane / 4 + 8 * r;
            if (h < s.heads) *reinterpret_cast<float2*>(out + (size_t)h * (s.cp + 2) + c) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
        }
    }
    if (tid < LD_HEADS && h0 + tid < s.heads) { out[(size_t)(h0 + tid) * (s.cp + 2) + s.cp] = mrow[tid]; out[(size_t)(h0 + tid) * (s.cp + 2) + s.cp + 1] = lrow[tid]; }
}

size_t decode_smem(const LatentShape& s) { return (size_t)(2 * LD_HEADS + LD_STAGES * LD_KEYS) * (s.cp + s.rp + 8) * 2; }

template <int NT>
cudaError_t decode_inst(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    const cudaError_t err = allow_smem(latent_decode_kernel<NT>, 216 * 1024, done);
    if (err != cudaSuccess) return err;
    return launch_pdl(latent_decode_kernel<NT>, dim3((a.s.heads + LD_HEADS - 1) / LD_HEADS, a.splits, tokens), dim3(256), decode_smem(a.s), st, pdl, a);
}

}  // namespace

bool latent_decode_fits(const LatentShape& s) { return s.cp <= 512 && decode_smem(s) <= 216 * 1024; }

cudaError_t launch_latent_decode(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (!latent_decode_fits(a.s) || !a.cache_bf16) return cudaErrorInvalidValue;
    if (a.s.cp <= 128) return decode_inst<2>(a, tokens, st, pdl);
    if (a.s.cp <= 256) return decode_inst<4>(a, tokens, st, pdl);
    return decode_inst<8>(a, tokens, st, pdl);
}

}  // namespace alice
