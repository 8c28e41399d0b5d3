// One head's rotation and norm, shared by the kernels of grouped attention.
#pragma once
#include "dense_dev.cuh"
#include "mixers.cuh"

namespace alice {

constexpr uint32_t GROUPED_PAIRS = GROUPED_MAX_DIM / 2;

// (cos, sin) of every rotated pair at position p; by the whole block of NT threads, without a barrier.
__device__ __forceinline__ void rotation_table(float2* cs, const float* freq, uint32_t half, uint32_t p, uint32_t nt) {
    for (uint32_t i = threadIdx.x; i < half; i += nt) {
        float sn, c;
        sincosf((float)p * freq[i], &sn, &c);
        cs[i] = make_float2(c, sn);
    }
}

// A warp takes one head's row x[0 .. dim) to out[0 .. dp): first rot_dims rotated half against half, then (unit) over the root
// of its mean square, zeros beyond dim. MAXE: elements a lane holds (32 * MAXE >= dp).
template <int MAXE, class OT>
__device__ __forceinline__ void rotate_norm_row(const float* x, OT* out, const GroupedShape& s, const float2* cs, float eps, uint32_t lane) {
    const uint32_t half = s.rot_dims / 2;
    float v[MAXE], q = 0.0f;
#pragma unroll
    for (int e = 0; e < MAXE; e++) {
        const uint32_t i = lane + 32 * e;
        v[e] = 0.0f;
        if (i >= s.dim) continue;
        v[e] = x[i];
        if (i < half) v[e] = v[e] * cs[i].x - x[i + half] * cs[i].y;
        else if (i < s.rot_dims) v[e] = v[e] * cs[i - half].x + x[i - half] * cs[i - half].y;
        q = fmaf(v[e], v[e], q);
    }
    float inv = 1.0f;
    if (s.unit_qk) inv = __frcp_rn(__fsqrt_rn(warp_sum(q) / (float)s.dim + eps));
#pragma unroll
    for (int e = 0; e < MAXE; e++)
        if (lane + 32 * e < s.dp) put(out + lane + 32 * e, v[e] * inv);
}
template <class OT>
__device__ __forceinline__ void rotate_norm(const float* x, OT* out, const GroupedShape& s, const float2* cs, float eps, uint32_t lane) {
    if (s.dp <= 64) rotate_norm_row<2>(x, out, s, cs, eps, lane);
    else if (s.dp <= 128) rotate_norm_row<4>(x, out, s, cs, eps, lane);
    else if (s.dp <= 256) rotate_norm_row<8>(x, out, s, cs, eps, lane);
    else rotate_norm_row<16>(x, out, s, cs, eps, lane);
}
// Value row, zeros beyond vdim.
template <class OT>
__device__ __forceinline__ void value_row(const float* x, OT* out, const GroupedShape& s, uint32_t lane) {
    for (uint32_t i = lane; i < s.vp; i += 32) put(out + i, i < s.vdim ? x[i] : 0.0f);
}

}  // namespace alice
