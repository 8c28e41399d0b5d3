// What the kernels of grouped attention share: the rotation table and one head's row with its rotation and norm.
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

// One head's row, held by a warp: lane l has elements l, l + 32, ... (E of them; 32 * E >= the padded length). Loading needs no
// position, so it can travel while the rotation table is made.
template <int E>
struct HeadRow {
    float v[E], other[E];   // other: the second of a rotated pair, where it does not lie in the same lane
    uint32_t n, rot;        // true length, rotated dimensions (0: a row that is only copied)

    __device__ __forceinline__ void load(const float* x, uint32_t n_, uint32_t rot_, uint32_t lane) {
        n = n_; rot = rot_;
        const uint32_t half = rot / 2;
#pragma unroll
        for (int e = 0; e < E; e++) {
            const uint32_t i = lane + 32 * e;
            v[e] = i < n ? __ldcg(x + i) : 0.0f;
            other[e] = half % 32 && i < rot ? __ldcg(x + (i < half ? i + half : i - half)) : 0.0f;
        }
    }
    template <int H>
    __device__ __forceinline__ void rotate_slots(const float2* cs, uint32_t lane) {   // half == 32 * H: pairs lie in one lane
#pragma unroll
        for (int e = 0; e < H && e + H < E; e++) {
            const float2 c = cs[lane + 32 * e];
            const float a = v[e], b = v[e + H];
            v[e] = a * c.x - b * c.y;
            v[e + H] = b * c.x + a * c.y;
        }
    }
    __device__ __forceinline__ void rotate(const float2* cs, uint32_t lane) {
        const uint32_t half = rot / 2;
        if (!half) return;
        if (half == 32) return rotate_slots<1>(cs, lane);
        if (half == 64) return rotate_slots<2>(cs, lane);
        if (half == 128) return rotate_slots<4>(cs, lane);
        if (half == 256) return rotate_slots<8>(cs, lane);
        if (half % 32) {
#pragma unroll
            for (int e = 0; e < E; e++) {
                const uint32_t i = lane + 32 * e;
                if (i < half) v[e] = v[e] * cs[i].x - other[e] * cs[i].y;
                else if (i < rot) v[e] = v[e] * cs[i - half].x + other[e] * cs[i - half].y;
            }
            return;
        }
#pragma unroll
        for (int h = 3; h < 8; h++)   // 96, 160, 192, 224
            if (half == 32u * h) {
                if (h == 3) rotate_slots<3>(cs, lane);
                else if (h == 5) rotate_slots<5>(cs, lane);
                else if (h == 6) rotate_slots<6>(cs, lane);
                else if (h == 7) rotate_slots<7>(cs, lane);
            }
    }
    // -> out[0 .. padded): rotated, over the root of its mean square where asked for, zeros beyond n
    template <class OT>
    __device__ __forceinline__ void store(OT* out, uint32_t padded, bool unit, const float2* cs, float eps, uint32_t lane) {
        rotate(cs, lane);
        float inv = 1.0f;
        if (unit) {
            float q = 0.0f;
#pragma unroll
            for (int e = 0; e < E; e++) q = fmaf(v[e], v[e], q);
            inv = __frcp_rn(__fsqrt_rn(warp_sum(q) / (float)n + eps));
        }
#pragma unroll
        for (int e = 0; e < E; e++)
            if (lane + 32 * e < padded) put(out + lane + 32 * e, v[e] * inv);
    }
};

}  // namespace alice
