// Causal attention of many tokens over rows of keys and values in global memory, on the tensor cores: bf16 queries, keys and
// values, f32 scores, softmax and sums. The softmax weights enter the weighted sum as a bf16 pair (value and remainder), so
// they are not cut to eight bits. The sink of a head is the state the online softmax starts from: a key that scores `sink`
// and has no value (-inf: no sink). Shared by the mixers that attend (latent_prefill.cu, grouped_prefill.cu).
#pragma once
#include "dense_dev.cuh"
#include "mixers.cuh"
#include "mma_sync.cuh"

namespace alice {

// Where the operands lie. Query head h reads key and value rows of head h / group; a key is k1's columns followed by k2's,
// which all heads share. Column counts are multiples of 8, rows 16-byte aligned.
struct PrefillArgs {
    uint32_t heads = 0, group = 1, vdim = 0, v_cols = 0;      // v_cols: vdim as the rows hold it
    const bf16* q = nullptr;                                  // rows of k1_cols + k2_cols, those of a group one behind the other
    size_t q_row = 0, q_group = 0;                            // elements between tokens and between groups
    const bf16 *k1 = nullptr, *k2 = nullptr, *v = nullptr;
    uint32_t k1_cols = 0, k2_cols = 0;
    size_t k1_row = 0, k1_head = 0, k2_row = 0, v_row = 0, v_head = 0;   // elements between rows and between heads
    const int* pos = nullptr;
    const float* sink = nullptr;
    float scale = 1.f, softcap = 0.f;                         // softcap 0: none (read by the CAP instances only)
    const float* gate = nullptr;                              // [t][ld_gate], sigmoid taken here; null: no gate
    uint32_t ld_gate = 0;
    bf16* out = nullptr;                                      // [t][ldo]: heads * vdim columns, zero up to ldo
    uint32_t ldo = 0;
};

constexpr int PF_KEYS = 32, PF_ROWS = 128, PF_THREADS = 128;   // keys per tile; queries per CTA, 32 per warp: each key fragment serves two row tiles

// DQ, DV: query / key and value dimensions the tiles have room for (multiples of 16, zero beyond the true sizes). Values wider
// than DV are cut into slices (blockIdx.z), each with its own pass over the scores.
template <int DQ, int DV>
struct PfGeom {
    static constexpr int LQ = DQ + 8, LV = DV + 8;   // row strides: eight rows land in different banks
    static constexpr size_t Q = (size_t)PF_ROWS * LQ * 2, K = (size_t)PF_KEYS * LQ * 2, V = (size_t)PF_KEYS * LV * 2, SMEM = Q + 2 * (K + V);
};

template <int DQ, int DV, bool CAP>
__global__ void __launch_bounds__(PF_THREADS, 2) attn_prefill_kernel(const __grid_constant__ PrefillArgs a, uint32_t tokens) {
    using G = PfGeom<DQ, DV>;
    extern __shared__ __align__(128) uint8_t sm[];
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x;
    const uint32_t t0 = (gridDim.y - 1 - blockIdx.y) * PF_ROWS;   // the longest rows first
    const uint32_t q_sm = smem_u32(sm), k_sm = q_sm + (uint32_t)G::Q, v_sm = k_sm + 2 * (uint32_t)G::K;
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t p0 = (uint32_t)*a.pos, qd = a.k1_cols + a.k2_cols;
    const uint32_t rows = min((uint32_t)PF_ROWS, tokens - t0), keys = p0 + t0 + rows, ntiles = (keys + PF_KEYS - 1) / PF_KEYS;
    const bf16 *k1 = a.k1 + (h / a.group) * a.k1_head, *v = a.v + (h / a.group) * a.v_head;
    const uint32_t v0 = blockIdx.z * DV, vn = min(a.v_cols - v0, (uint32_t)DV);   // this slice of the values

    // zero what lies beyond the true sizes once (the copies below never touch it)
    for (uint32_t i = tid; i < 2 * PF_KEYS * (DQ - qd); i += PF_THREADS) {
        const uint32_t r = i / (DQ - qd), c = qd + i % (DQ - qd);
        reinterpret_cast<bf16*>(sm + G::Q + (r / PF_KEYS) * G::K)[(r % PF_KEYS) * G::LQ + c] = __float2bfloat16_rn(0.0f);
    }
    for (uint32_t i = tid; i < 2 * PF_KEYS * (DV - vn); i += PF_THREADS) {
        const uint32_t r = i / (DV - vn), c = vn + i % (DV - vn);
        reinterpret_cast<bf16*>(sm + G::Q + 2 * G::K + (r / PF_KEYS) * G::V)[(r % PF_KEYS) * G::LV + c] = __float2bfloat16_rn(0.0f);
    }
    // rows of 16-byte pieces, a few threads a row
    constexpr uint32_t TPR = PF_THREADS / PF_KEYS;
    const uint32_t fr = tid / TPR, fc = tid % TPR, nd = a.k1_cols / 8, nr = a.k2_cols / 8, nv = vn / 8;
    auto fetch = [&](uint32_t tile, uint32_t b) {
        const uint32_t j = min(tile * PF_KEYS + fr, keys - 1);
        const bool ok = tile * PF_KEYS + fr < keys;
        const uint32_t kd = k_sm + b * (uint32_t)G::K + fr * G::LQ * 2, vd = v_sm + b * (uint32_t)G::V + fr * G::LV * 2;
        const bf16 *kp = k1 + j * a.k1_row, *rp = a.k2 + j * a.k2_row, *vp = v + j * a.v_row + v0;
        for (uint32_t c = fc; c < nd; c += TPR) cp16(kd + c * 16, kp + c * 8, ok);
        for (uint32_t c = fc; c < nr; c += TPR) cp16(kd + (nd + c) * 16, rp + c * 8, ok);
        for (uint32_t c = fc; c < nv; c += TPR) cp16(vd + c * 16, vp + c * 8, ok);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (uint32_t r = fr; r < PF_ROWS; r += PF_KEYS) {   // queries, part of the first copy group
        const bf16* q = a.q + (t0 + min(r, rows - 1)) * a.q_row + (h / a.group) * a.q_group + (h % a.group) * qd;
        for (uint32_t c = fc; c < DQ / 8; c += TPR) cp16(q_sm + r * G::LQ * 2 + c * 16, q + min(c * 8, qd - 8), r < rows && c * 8 < qd);
    }
    fetch(0, 0);

    // a thread's rows are lane / 4 and lane / 4 + 8 of each of its warp's two 16-row tiles
    constexpr float LOG2E = 1.4426950408889634f;
    const float scale = CAP && a.softcap > 0.0f ? a.scale / a.softcap * 2.0f * LOG2E : a.scale * LOG2E;   // with a cap: to 2 s / cap in powers of two
    const float cap = a.softcap * LOG2E;
    float m[2][2], l[2][2], o[2][DV / 8][4];
#pragma unroll
    for (int g = 0; g < 2; g++) {
        m[g][0] = m[g][1] = a.sink[h] * LOG2E;
        l[g][0] = l[g][1] = (lane & 3) == 0 ? 1.0f : 0.0f;
#pragma unroll
        for (int i = 0; i < DV / 8; i++) o[g][i][0] = o[g][i][1] = o[g][i][2] = o[g][i][3] = 0.0f;
    }
    const uint32_t row0 = warp * 32 + lane / 4, see = p0 + t0 + row0;   // last key the first of them sees
    const uint32_t q_addr = q_sm + ((warp * 32 + lane % 16) * G::LQ + lane / 16 * 8) * 2;

    for (uint32_t tile = 0; tile < ntiles; tile++) {
        const uint32_t b = tile & 1;
        if (tile + 1 < ntiles) {
            fetch(tile + 1, b ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t kt = k_sm + b * (uint32_t)G::K, vt = v_sm + b * (uint32_t)G::V;
        float sc[2][PF_KEYS / 8][4];
#pragma unroll
        for (int g = 0; g < 2; g++)
#pragma unroll
            for (int i = 0; i < PF_KEYS / 8; i++) sc[g][i][0] = sc[g][i][1] = sc[g][i][2] = sc[g][i][3] = 0.0f;
        const uint32_t k_addr = kt + ((lane % 8 + lane / 16 * 8) * G::LQ + (lane / 8 % 2) * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < DQ / 16; kk++) {
            uint32_t q0[4], q1[4];
            ldsm4(q0, q_addr + kk * 32);
            ldsm4(q1, q_addr + 16 * G::LQ * 2 + kk * 32);
#pragma unroll
            for (int n = 0; n < PF_KEYS / 16; n++) {
                uint32_t kb[4];
                ldsm4(kb, k_addr + (n * 16 * G::LQ + kk * 16) * 2);
                mma16816(sc[0][2 * n], q0, kb[0], kb[1]);
                mma16816(sc[0][2 * n + 1], q0, kb[2], kb[3]);
                mma16816(sc[1][2 * n], q1, kb[0], kb[1]);
                mma16816(sc[1][2 * n + 1], q1, kb[2], kb[3]);
            }
        }
        const uint32_t j0 = tile * PF_KEYS + (lane & 3) * 2;
        const bool edge = tile * PF_KEYS + PF_KEYS > p0 + t0 + warp * 32;   // some key of the tile is hidden from some row of the warp
#pragma unroll
        for (int g = 0; g < 2; g++) {
            float top0 = m[g][0], top1 = m[g][1];
#pragma unroll
            for (int i = 0; i < PF_KEYS / 8; i++) {
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    float v = sc[g][i][e] * scale;
                    if (CAP && a.softcap > 0.0f) v = cap * tanh_of_pow2(v);
                    if (edge && j0 + i * 8 + (e & 1) > see + g * 16 + (e < 2 ? 0 : 8)) v = -INFINITY;
                    sc[g][i][e] = v;
                }
                top0 = fmaxf(top0, fmaxf(sc[g][i][0], sc[g][i][1]));
                top1 = fmaxf(top1, fmaxf(sc[g][i][2], sc[g][i][3]));
            }
#pragma unroll
            for (int x = 1; x <= 2; x *= 2) {
                top0 = fmaxf(top0, __shfl_xor_sync(0xffffffffu, top0, x));
                top1 = fmaxf(top1, __shfl_xor_sync(0xffffffffu, top1, x));
            }
            const float f0 = exp2f(m[g][0] - top0), f1 = exp2f(m[g][1] - top1);
            if (__any_sync(0xffffffffu, f0 != 1.0f || f1 != 1.0f)) {
#pragma unroll
                for (int i = 0; i < DV / 8; i++) { o[g][i][0] *= f0; o[g][i][1] *= f0; o[g][i][2] *= f1; o[g][i][3] *= f1; }
            }
            m[g][0] = top0; m[g][1] = top1;
            l[g][0] *= f0; l[g][1] *= f1;
#pragma unroll
            for (int i = 0; i < PF_KEYS / 8; i++) {
                sc[g][i][0] = exp2f(sc[g][i][0] - top0); sc[g][i][1] = exp2f(sc[g][i][1] - top0);
                sc[g][i][2] = exp2f(sc[g][i][2] - top1); sc[g][i][3] = exp2f(sc[g][i][3] - top1);
                l[g][0] += sc[g][i][0] + sc[g][i][1]; l[g][1] += sc[g][i][2] + sc[g][i][3];
            }
        }
        const uint32_t v_addr = vt + ((lane % 16) * G::LV + lane / 16 * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < PF_KEYS / 16; kk++) {
            uint32_t hi[2][4], lo[2][4];
#pragma unroll
            for (int g = 0; g < 2; g++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float x = sc[g][2 * kk + e / 2][(e & 1) * 2], y = sc[g][2 * kk + e / 2][(e & 1) * 2 + 1];
                    hi[g][e] = pack_bf16(x, y);
                    const float2 r = bf2(hi[g][e]);
                    lo[g][e] = pack_bf16(x - r.x, y - r.y);
                }
#pragma unroll
            for (int n = 0; n < DV / 16; n++) {
                uint32_t vb[4];
                ldsm4t(vb, v_addr + (kk * 16 * G::LV + n * 16) * 2);
#pragma unroll
                for (int g = 0; g < 2; g++) {
                    mma16816(o[g][2 * n], hi[g], vb[0], vb[1]);
                    mma16816(o[g][2 * n + 1], hi[g], vb[2], vb[3]);
                    mma16816(o[g][2 * n], lo[g], vb[0], vb[1]);
                    mma16816(o[g][2 * n + 1], lo[g], vb[2], vb[3]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int g = 0; g < 2; g++)
#pragma unroll
        for (int r = 0; r < 2; r++) {
            float den = l[g][r];
            den += __shfl_xor_sync(0xffffffffu, den, 1);
            den += __shfl_xor_sync(0xffffffffu, den, 2);
            const float inv = __frcp_rn(den);
            const uint32_t row = row0 + 16 * g + 8 * r;
            if (row >= rows) continue;
            bf16* out = a.out + (size_t)(t0 + row) * a.ldo + (size_t)h * a.vdim + v0;
            const float* gate = a.gate ? a.gate + (size_t)(t0 + row) * a.ld_gate + (size_t)h * a.vdim + v0 : nullptr;
            const uint32_t n = min(a.vdim - v0, (uint32_t)DV);
#pragma unroll
            for (int i = 0; i < DV / 8; i++) {
                const uint32_t c = i * 8 + (lane & 3) * 2;
                if (c >= n) continue;
                float x = o[g][i][2 * r] * inv, y = o[g][i][2 * r + 1] * inv;
                if (gate) { x *= sigmoid_f(gate[c]); y *= c + 1 < n ? sigmoid_f(gate[c + 1]) : 0.0f; }
                if (a.vdim % 2 == 0) {
                    *reinterpret_cast<uint32_t*>(out + c) = pack_bf16(x, y);
                } else {
                    put(out + c, x);
                    if (c + 1 < n) put(out + c + 1, y);
                }
            }
            if (h + 1 == a.heads && blockIdx.z == 0)   // padding up to the stride
                for (uint32_t c = a.vdim + (lane & 3); c < a.ldo - h * a.vdim; c += 4) out[c] = __float2bfloat16_rn(0.0f);
        }
}

template <int DQ, int DV, bool CAP>
cudaError_t attn_prefill_inst(const PrefillArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    const cudaError_t err = allow_smem(attn_prefill_kernel<DQ, DV, CAP>, PfGeom<DQ, DV>::SMEM, done);
    if (err != cudaSuccess) return err;
    return launch_pdl(attn_prefill_kernel<DQ, DV, CAP>, dim3(a.heads, (tokens + PF_ROWS - 1) / PF_ROWS, (a.v_cols + DV - 1) / DV), dim3(PF_THREADS),
                      PfGeom<DQ, DV>::SMEM, st, pdl, a, tokens);
}
template <bool CAP>
cudaError_t launch_attn_prefill(const PrefillArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    const uint32_t q = a.k1_cols + a.k2_cols, v = a.v_cols;
    if (!tokens || q > 256 || v > 256 || (a.k1_cols | a.k2_cols | v) % 8 || a.heads % a.group) return cudaErrorInvalidValue;
    if (q <= 64 && v <= 64) return attn_prefill_inst<64, 64, CAP>(a, tokens, st, pdl);
    if (q <= 64 && v <= 128) return attn_prefill_inst<64, 128, CAP>(a, tokens, st, pdl);
    if (q <= 128 && v <= 128) return attn_prefill_inst<128, 128, CAP>(a, tokens, st, pdl);
    if (q <= 192) return attn_prefill_inst<192, 128, CAP>(a, tokens, st, pdl);
    return attn_prefill_inst<256, 128, CAP>(a, tokens, st, pdl);
}

}  // namespace alice
