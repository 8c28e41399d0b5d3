// Grouped attention of one to a few tokens over a bfloat16 cache on the tensor cores. Up to sixteen query heads of a group are
// the rows of one product with the keys they share. The context is dealt to CTAs in shares and within a CTA to its warps in
// tiles of sixteen keys; each warp streams its own tiles with bulk copies through a ring of its own, so no warp waits for
// another until the sums are joined. The CTA that finishes a group of heads last joins the shares and the sink.
#include "grouped_dev.cuh"
#include "mma_sync.cuh"

namespace alice {
namespace {

constexpr uint32_t GD_HEADS = 16, GD_KEYS = GROUPED_TILE, GD_WARPS = 8, GD_MAX_STAGES = 4, GD_MAX_SPLITS = 160;
constexpr int KERR_GROUPED_WAIT = 8;   // a copied tile of keys and values did not arrive
constexpr size_t GD_SMEM = 200 * 1024;

// Geometry both sides use: dynamic shared memory is [16][dp + 8] queries, then warps * stages tiles of [16][ld].
struct GdGeom {
    uint32_t warps, stages;
    size_t smem;
};
GdGeom gd_geom(const GroupedShape& s) {
    GdGeom g;
    const size_t q = (size_t)GD_HEADS * (s.dp + 8) * 2, tile = (size_t)GD_KEYS * s.ld() * 2;
    for (g.warps = GD_WARPS;; g.warps /= 2) {
        g.stages = (uint32_t)std::min<size_t>(GD_MAX_STAGES, (GD_SMEM - q) / (tile * g.warps));
        if (g.stages >= 2 || g.warps == 1) break;
    }
    g.smem = q + tile * g.warps * g.stages + 128;
    return g;
}

// grid (kv_heads * groups of 16 heads, splits, tokens). NT: 8-column tiles of the weighted sum (8 * NT >= vp).
template <int NT, class OT>
__global__ void __launch_bounds__(GD_WARPS * 32, 1) grouped_decode_kernel(const __grid_constant__ GroupedArgs a, uint32_t stages) {
    extern __shared__ uint8_t raw[];
    __shared__ __align__(8) uint64_t bars[GD_WARPS][GD_MAX_STAGES];
    __shared__ float2 cs[128];
    __shared__ float wm[GD_WARPS][GD_HEADS], wl[GD_WARPS][GD_HEADS], wt[GD_HEADS][GD_MAX_SPLITS];
    __shared__ unsigned int last_one;
    const GroupedShape& s = a.s;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, W = blockDim.x >> 5, t = blockIdx.z;
    const uint32_t group = s.heads / s.kv_heads, hg = (group + GD_HEADS - 1) / GD_HEADS;
    const uint32_t kh = blockIdx.x / hg, h0 = kh * group + blockIdx.x % hg * GD_HEADS, rows = min(GD_HEADS, group - blockIdx.x % hg * GD_HEADS);
    const uint32_t ld = s.ld(), tile_bytes = GD_KEYS * ld * 2, ldq = s.dp + 8;
    uint8_t* base = raw + (128 - (smem_u32(raw) & 127)) % 128;
    auto* qs = reinterpret_cast<bf16*>(base);
    uint8_t* ring = base + GD_HEADS * ldq * 2;
    const uint32_t q_sm = smem_u32(qs), ring_sm = smem_u32(ring) + warp * stages * tile_bytes;
    pdl_launch_dependents();
    if (lane == 0) {
        for (uint32_t i = 0; i < stages; i++) mbar_init(smem_u32(&bars[warp][i]), 1);
        mbar_fence_init();
    }
    __syncwarp();
    pdl_wait();
    // rows that need no position travel together with it
    const float* y = a.y + (size_t)t * a.ldy;
    HeadRow<8> query, key, value;
    if (warp < rows) query.load(y + (size_t)(h0 + warp) * s.dim, s.dim, s.rot_dims, lane);
    if (a.append && warp == W - 1) {
        key.load(y + s.off_k + (size_t)kh * s.dim, s.dim, s.rot_dims, lane);
        value.load(y + s.off_v + (size_t)kh * s.vdim, s.vdim, 0, lane);
    }
    const uint32_t pos = (uint32_t)*a.pos + t, ctx = pos + 1, tiles = (ctx + GD_KEYS - 1) / GD_KEYS;
    const uint32_t per = ((tiles + gridDim.y - 1) / gridDim.y + W - 1) / W * W, shares = (tiles + per - 1) / per;
    const uint32_t lo = blockIdx.y * per, hi = min(tiles, lo + per);
    if (lo >= hi) return;   // the whole CTA: this share is not among those that are joined
    const size_t plane = (size_t)kh * a.plane_rows * ld;
    const bf16* keys = static_cast<const bf16*>(a.cache) + plane;
    const bool fresh = a.append && hi == tiles;       // this CTA makes the token's own row; it lies in the last tile
    const uint32_t mine = lo + warp < hi ? (hi - lo - warp + W - 1) / W : 0;   // tiles of this warp
    auto issue = [&](uint32_t i) {
        if (lane == 0) {
            const uint32_t bar = smem_u32(&bars[warp][i % stages]);
            mbar_arrive_expect_tx(bar, tile_bytes);
            bulk_g2s(ring_sm + i % stages * tile_bytes, keys + (size_t)(lo + warp + i * W) * GD_KEYS * ld, tile_bytes, bar);
        }
    };
    uint32_t issued = 0;
    for (; issued < min(stages, mine); issued++) {
        if (fresh && lo + warp + issued * W == tiles - 1) break;
        issue(issued);
    }
    const uint32_t half = s.rot_dims / 2;
    rotation_table(cs, a.freq, half, pos, blockDim.x);
    __syncthreads();
    if (fresh && warp == W - 1) {
        bf16* out = static_cast<bf16*>(a.cache) + plane + (size_t)pos * ld;
        key.store(out, s.dp, s.unit_qk, cs, a.eps, lane);   // further head groups of these keys write the same bits
        value.store(out + s.dp, s.vp, false, cs, a.eps, lane);
        __threadfence();
        asm volatile("fence.proxy.async.global;" ::: "memory");   // the bulk copy below reads what this warp has written
    }
    for (uint32_t r = warp; r < GD_HEADS; r += W) {
        if (r < rows) {
            if (r >= W) query.load(y + (size_t)(h0 + r) * s.dim, s.dim, s.rot_dims, lane);
            query.store(qs + r * ldq, s.dp, s.unit_qk, cs, a.eps, lane);
        } else {
            for (uint32_t i = lane; i < s.dp; i += 32) put(qs + r * ldq + i, 0.0f);
        }
    }
    __syncthreads();
    for (; issued < min(stages, mine); issued++) issue(issued);

    constexpr float LOG2E = 1.4426950408889634f;
    // scores in powers of two; bounded ones need no running maximum
    const bool bounded = a.bounded;
    const float scale = s.softcap > 0.0f ? s.scale / s.softcap * 2.0f * LOG2E : s.scale * LOG2E, cap = s.softcap * LOG2E;
    float m[2], l[2] = {0.0f, 0.0f}, o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    m[0] = m[1] = bounded ? 0.0f : -INFINITY;
    const uint32_t q_addr = q_sm + ((lane % 16) * ldq + lane / 16 * 8) * 2;
    uint32_t done = 0;
    for (; done < mine; done++) {
        const uint32_t slot = done % stages, k0 = (lo + warp + done * W) * GD_KEYS, kb = ring_sm + slot * tile_bytes;
        const bool ok = mbar_wait(smem_u32(&bars[warp][slot]), (done / stages) & 1);
        if (!__all_sync(0xffffffffu, ok)) { if (lane == 0) atomicCAS(a.status, 0, KERR_GROUPED_WAIT); break; }
        float d[2][2][4] = {};   // two chains per tile of eight keys
        const uint32_t k_addr = kb + ((lane % 8 + lane / 16 * 8) * ld + (lane / 8 % 2) * 8) * 2;
#pragma unroll 4
        for (uint32_t kk = 0; kk < s.dp / 16; kk++) {
            uint32_t q4[4], k4[4];
            ldsm4(q4, q_addr + kk * 32);
            ldsm4(k4, k_addr + kk * 32);
            if (kk & 1) { mma16816(d[1][0], q4, k4[0], k4[1]); mma16816(d[1][1], q4, k4[2], k4[3]); }
            else { mma16816(d[0][0], q4, k4[0], k4[1]); mma16816(d[0][1], q4, k4[2], k4[3]); }
        }
        float sc[2][4], top0 = m[0], top1 = m[1];
#pragma unroll
        for (int n = 0; n < 2; n++) {
#pragma unroll
            for (int e = 0; e < 4; e++) {
                float v = (d[0][n][e] + d[1][n][e]) * scale;
                if (s.softcap > 0.0f) v = cap * tanh_of_pow2(v);
                sc[n][e] = k0 + n * 8 + (lane & 3) * 2 + (e & 1) < ctx ? v : -INFINITY;
            }
            top0 = fmaxf(top0, fmaxf(sc[n][0], sc[n][1]));
            top1 = fmaxf(top1, fmaxf(sc[n][2], sc[n][3]));
        }
        if (!bounded) {
#pragma unroll
            for (int x = 1; x <= 2; x *= 2) {
                top0 = fmaxf(top0, __shfl_xor_sync(0xffffffffu, top0, x));
                top1 = fmaxf(top1, __shfl_xor_sync(0xffffffffu, top1, x));
            }
            const float f0 = exp2f(m[0] - top0), f1 = exp2f(m[1] - top1);   // a tile holds at least one key: the tops are finite
            m[0] = top0; m[1] = top1;
            l[0] *= f0; l[1] *= f1;
#pragma unroll
            for (int i = 0; i < NT; i++) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
        }
        uint32_t hi4[4], lo4[4];
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const float tp = m[e & 1];
            const float x = exp2f(sc[e / 2][(e & 1) * 2] - tp), z = exp2f(sc[e / 2][(e & 1) * 2 + 1] - tp);
            l[e & 1] += x + z;
            hi4[e] = pack_bf16(x, z);
            const float2 r = bf2(hi4[e]);
            lo4[e] = pack_bf16(x - r.x, z - r.y);
        }
        const uint32_t v_addr = kb + ((lane % 16) * ld + s.dp + lane / 16 * 8) * 2;
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
            if (n * 8 >= (int)s.vp) break;   // vp is a multiple of 16: whole pairs of tiles
            uint32_t v4[4];
            ldsm4t(v4, v_addr + n * 16);
            mma16816(o[n], hi4, v4[0], v4[1]);
            mma16816(o[n + 1], hi4, v4[2], v4[3]);
            mma16816(o[n], lo4, v4[0], v4[1]);
            mma16816(o[n + 1], lo4, v4[2], v4[3]);
        }
        __syncwarp();
        if (issued < mine) issue(issued++);
    }
    for (; done < issued; done++) mbar_wait(smem_u32(&bars[warp][done % stages]), (done / stages) & 1);   // only after a wait that ran out

    // the warps' sums meet in the ring's place
#pragma unroll
    for (int r = 0; r < 2; r++) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        if ((lane & 3) == 0) { wm[warp][lane / 4 + 8 * r] = m[r]; wl[warp][lane / 4 + 8 * r] = l[r]; }
    }
    __syncthreads();
    auto* comb = reinterpret_cast<float*>(ring);     // [W][rows][vp]: at most warps * 16 * vp * 4 bytes of the ring's warps * stages * 16 * ld * 2
    const uint32_t vp = s.vp, stride = vp + 4;
#pragma unroll
    for (int i = 0; i < NT; i++) {
        const uint32_t c = i * 8 + (lane & 3) * 2;
        if (c >= vp) break;
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const uint32_t row = lane / 4 + 8 * r;
            if (row < rows) *reinterpret_cast<float2*>(comb + ((size_t)warp * rows + row) * vp + c) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
        }
    }
    __syncthreads();
    float* part = a.part + (size_t)t * gridDim.y * s.heads * stride;
    for (uint32_t i = tid; i < rows * vp; i += blockDim.x) {
        const uint32_t r = i / vp, c = i % vp;
        float top = -INFINITY;
        for (uint32_t w = 0; w < W; w++) top = fmaxf(top, wm[w][r]);
        float v = 0.0f, den = 0.0f;
        for (uint32_t w = 0; w < W; w++) {
            const float f = exp2f(wm[w][r] - top);   // 0 for a warp without tiles
            v = fmaf(f, comb[((size_t)w * rows + r) * vp + c], v);
            den = fmaf(f, wl[w][r], den);
        }
        float* out = part + ((size_t)blockIdx.y * s.heads + h0 + r) * stride;
        out[4 + c] = v;
        if (c == 0) { out[0] = top; out[1] = den; }
    }
    __threadfence();
    __syncthreads();
    unsigned int* ticket = a.tickets + (size_t)t * gridDim.x + blockIdx.x;
    if (tid == 0) last_one = atomicAdd(ticket, 1u) == shares - 1;
    __syncthreads();
    if (!last_one) return;
    if (tid == 0) *ticket = 0;   // for the next launch
    __threadfence();
    for (uint32_t r = warp; r < rows; r += W) {
        const float sink = a.sink[h0 + r] * LOG2E;
        const float* p = part + (size_t)(h0 + r) * stride;
        const size_t step = (size_t)s.heads * stride;
        float top = sink;
        for (uint32_t k = lane; k < shares; k += 32) top = fmaxf(top, __ldcg(p + k * step));
        top = warp_max(top);
        float den = 0.0f;
        for (uint32_t k = lane; k < shares; k += 32) {
            const float f = exp2f(__ldcg(p + k * step) - top);
            wt[r][k] = f;
            den = fmaf(f, __ldcg(p + k * step + 1), den);
        }
        den = warp_sum(den) + exp2f(sink - top);
        const float inv = __frcp_rn(den);
        for (uint32_t k = lane; k < shares; k += 32) wt[r][k] *= inv;
    }
    __syncthreads();
    OT* out = static_cast<OT*>(a.out) + (size_t)t * a.ldo + (size_t)h0 * s.vdim;
    for (uint32_t i = tid; i < rows * s.vdim; i += blockDim.x) {
        const uint32_t r = i / s.vdim, c = i % s.vdim;
        const float* p = part + (size_t)(h0 + r) * stride + 4 + c;
        const size_t step = (size_t)s.heads * stride;
        float v = 0.0f;
#pragma unroll 16
        for (uint32_t k = 0; k < shares; k++) v = fmaf(wt[r][k], __ldcg(p + k * step), v);
        put(out + (size_t)r * s.vdim + c, v);
    }
    if (h0 + rows == s.heads)   // padding up to the stride
        for (uint32_t c = rows * s.vdim + tid; c < a.ldo - h0 * s.vdim; c += blockDim.x) put(out + c, 0.0f);
}

template <int NT, class OT>
cudaError_t decode_inst(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    const cudaError_t err = allow_smem(grouped_decode_kernel<NT, OT>, 208 * 1024, done);
    if (err != cudaSuccess) return err;
    const GdGeom g = gd_geom(a.s);
    const uint32_t hg = (a.s.group() + GD_HEADS - 1) / GD_HEADS;
    return launch_pdl(grouped_decode_kernel<NT, OT>, dim3(a.s.kv_heads * hg, a.splits, tokens), dim3(g.warps * 32), g.smem, st, pdl, a, g.stages);
}
template <class OT>
cudaError_t decode_type(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (a.s.vp <= 64) return decode_inst<8, OT>(a, tokens, st, pdl);
    if (a.s.vp <= 128) return decode_inst<16, OT>(a, tokens, st, pdl);
    return decode_inst<32, OT>(a, tokens, st, pdl);
}

}  // namespace

cudaError_t launch_grouped_decode(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl) {
    if (!grouped_tiled_fits(a.s) || !a.cache_bf16 || !a.splits || a.splits > GD_MAX_SPLITS || (a.append && tokens != 1) || gd_geom(a.s).stages < 2)
        return cudaErrorInvalidValue;
    return a.act_bf16 ? decode_type<bf16>(a, tokens, st, pdl) : decode_type<float>(a, tokens, st, pdl);
}

}  // namespace alice
