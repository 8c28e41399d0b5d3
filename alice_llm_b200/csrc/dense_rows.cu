// One token against dense bfloat16 rows. A warp owns R consecutive rows at a time; every lane requests 16-byte pieces in batches
// of R * 8, so two CTAs of eight warps per SM keep enough bytes in flight and leave room for the CTAs of the next kernel. The
// input sits in shared memory as f32. The beginning of the rows a warp starts with is requested into L2 before the wait for the
// producing kernel (a longer prefetch made the stream slower: 4096 x 18432 in 28.7 us without, 34.9 us with whole rows).
#include "dense_dev.cuh"

namespace alice {
namespace {

constexpr int RT = 256, RW = RT / 32;

template <int R, int U>
__device__ __forceinline__ void dot_batches(const bf16* const (&w)[R], const float* xs, uint32_t& c, uint32_t k, float (&acc)[R]) {
    for (; c + (U - 1) * 256 < k; c += U * 256) {
        uint4 v[U][R];
#pragma unroll
        for (int u = 0; u < U; u++)
#pragma unroll
            for (int r = 0; r < R; r++) v[u][r] = __ldg(reinterpret_cast<const uint4*>(w[r] + c + u * 256));
#pragma unroll
        for (int u = 0; u < U; u++) {
            const float4 x0 = *reinterpret_cast<const float4*>(xs + c + u * 256), x1 = *reinterpret_cast<const float4*>(xs + c + u * 256 + 4);
#pragma unroll
            for (int r = 0; r < R; r++) acc[r] = dot8(v[u][r], x0, x1, acc[r]);
        }
    }
}
// acc[r] = w[r][0 .. k) . xs[0 .. k), the same in every lane
template <int R>
__device__ __forceinline__ void dot_rows(const bf16* const (&w)[R], const float* xs, uint32_t k, uint32_t lane, float (&acc)[R]) {
#pragma unroll
    for (int r = 0; r < R; r++) acc[r] = 0.0f;
    uint32_t c = lane * 8;
    dot_batches<R, 8>(w, xs, c, k, acc);
    dot_batches<R, 4>(w, xs, c, k, acc);
    dot_batches<R, 2>(w, xs, c, k, acc);
    dot_batches<R, 1>(w, xs, c, k, acc);
#pragma unroll
    for (int r = 0; r < R; r++) acc[r] = warp_sum(acc[r]);
}

__device__ __forceinline__ void prefetch_row(const bf16* w, uint32_t k, uint32_t lane) {
    if (lane * 64 < k) prefetch_l2(w + lane * 64);
}

// order-preserving image of a float, as the output head's argmax packs it
__device__ __forceinline__ unsigned long long argmax_pack(float v, uint32_t row) {
    uint32_t u = __float_as_uint(v);
    u = (u & 0x80000000u) ? ~u : (u | 0x80000000u);
    return ((unsigned long long)u << 32) | (0xFFFFFFFFu - row);
}

// Item i of the work list: R rows of w0, or R / 2 gate rows with their up rows.
template <int R>
__device__ __forceinline__ void item_rows(const RowsIn& op, uint32_t item, uint32_t items0, const bf16* (&w)[R], uint32_t& first, bool& pair) {
    pair = item >= items0;
    if (!pair) {
        first = item * R;
#pragma unroll
        for (int r = 0; r < R; r++) w[r] = op.w0.w + (size_t)min(first + r, op.w0.n - 1) * op.w0.k;
    } else {
        first = (item - items0) * (R / 2);
#pragma unroll
        for (int r = 0; r < R / 2; r++) {
            const uint32_t c = first + r, row = (c / 64) * 128 + c % 64;
            w[r] = op.gu.w + (size_t)row * op.gu.k;
            w[R / 2 + r] = w[r] + (size_t)64 * op.gu.k;
        }
    }
}

template <int R>
__global__ void __launch_bounds__(RT, 2) rows_in_kernel(const __grid_constant__ RowsIn op) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float red[RW];
    const uint32_t lane = threadIdx.x & 31, warps = gridDim.x * RW;
    const uint32_t items0 = (op.w0.n + R - 1) / R, items = items0 + op.gu.n / R;
    const uint32_t w_id = blockIdx.x + (threadIdx.x >> 5) * gridDim.x;
    const uint32_t k = op.w0.n ? op.w0.k : op.gu.k;
    const bf16* w[R];
    uint32_t first;
    bool pair;
    pdl_launch_dependents();
    if (w_id < items) {
        item_rows<R>(op, w_id, items0, w, first, pair);
#pragma unroll
        for (int r = 0; r < R; r++) prefetch_row(w[r], k, lane);
    }
    pdl_wait();
    load_normed<RW>(xs, op.x, op.n_x, k, op.norm, op.norm_w, op.eps, red);
    if (op.h_out && blockIdx.x == 0)
        for (uint32_t i = threadIdx.x; i < op.n_x; i += RT) op.h_out[i] = xs[i];
    unsigned long long best = 0ull;
    for (uint32_t item = w_id; item < items; item += warps) {
        item_rows<R>(op, item, items0, w, first, pair);
        float acc[R];
        dot_rows<R>(w, xs, k, lane, acc);
        if (!pair) {
#pragma unroll
            for (int r = 0; r < R; r++) {
                if (first + r >= op.w0.n) break;
                if (lane == (uint32_t)r) op.y0[first + r] = acc[r];
                if (op.argmax_key) { const unsigned long long key = argmax_pack(acc[r], first + r); best = key > best ? key : best; }
            }
        } else {
#pragma unroll
            for (int r = 0; r < R / 2; r++)
                if (lane == (uint32_t)r) {
                    const float g = op.gate_b ? acc[r] + op.gate_b[first + r] : acc[r], u = op.up_b ? acc[R / 2 + r] + op.up_b[first + r] : acc[R / 2 + r];
                    op.y1[first + r] = silu_ref(g) * u;
                }
        }
    }
    if (op.argmax_key && lane == 0 && best) atomicMax(op.argmax_key, best);
}

template <int R>
__global__ void __launch_bounds__(RT, 2) rows_out_kernel(const __grid_constant__ RowsOut op) {
    extern __shared__ __align__(16) float xs[];
    const uint32_t lane = threadIdx.x & 31, warps = gridDim.x * RW, w_id = blockIdx.x + (threadIdx.x >> 5) * gridDim.x;
    const uint32_t n = op.w1.n, k1 = op.w1.k, k2 = op.w2.n ? op.w2.k : 0, items = (n + R - 1) / R;
    pdl_launch_dependents();
    if (w_id < items)
#pragma unroll
        for (int r = 0; r < R; r++) {
            const uint32_t row = min(w_id * R + r, n - 1);
            prefetch_row(op.w1.w + (size_t)row * k1, k1, lane);
            if (k2) prefetch_row(op.w2.w + (size_t)row * k2, k2, lane);
        }
    pdl_wait();
    for (uint32_t i = threadIdx.x * 4; i < k1; i += RT * 4) *reinterpret_cast<float4*>(xs + i) = __ldcg(reinterpret_cast<const float4*>(op.a + i));
    for (uint32_t i = threadIdx.x * 4; i < k2; i += RT * 4) *reinterpret_cast<float4*>(xs + k1 + i) = __ldcg(reinterpret_cast<const float4*>(op.f + i));
    __syncthreads();
    for (uint32_t item = w_id; item < items; item += warps) {
        const bf16 *u[R], *d[R];
#pragma unroll
        for (int r = 0; r < R; r++) {
            const uint32_t row = min(item * R + r, n - 1);
            u[r] = op.w1.w + (size_t)row * k1;
            d[r] = op.w2.w + (size_t)row * k2;
        }
        float acc1[R], acc2[R];
#pragma unroll
        for (int r = 0; r < R; r++) acc2[r] = 0.0f;
        if (k2) dot_rows<R>(d, xs + k1, k2, lane, acc2);
        dot_rows<R>(u, xs, k1, lane, acc1);
#pragma unroll
        for (int r = 0; r < R; r++) {
            const uint32_t row = item * R + r;
            if (lane == (uint32_t)r && row < n) {
                float v = op.s1 ? op.s1[row] * acc1[r] : acc1[r];
                if (k2) v += op.s2[row] * (acc2[r] + op.b2[row]);
                op.out[row] = op.alpha * op.x[row] + v;
            }
        }
    }
}

template <int R>
cudaError_t rows_out_r(const RowsOut& op, int num_sms, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    const cudaError_t err = allow_smem(rows_out_kernel<R>, 224 * 1024, done);
    if (err != cudaSuccess) return err;
    const uint32_t items = (op.w1.n + R - 1) / R, grid = std::min<uint32_t>((items + RW - 1) / RW, (uint32_t)num_sms * 2);
    return launch_pdl(rows_out_kernel<R>, dim3(grid), dim3(RT), (size_t)(op.w1.k + (op.w2.n ? op.w2.k : 0)) * 4, st, pdl, op);
}

template <int R>
cudaError_t rows_in_r(const RowsIn& op, int num_sms, cudaStream_t st, bool pdl) {
    static bool done[64] = {};
    cudaError_t err = allow_smem(rows_in_kernel<R>, 224 * 1024, done);
    if (err != cudaSuccess) return err;
    const uint32_t items = (op.w0.n + R - 1) / R + op.gu.n / R;
    const uint32_t grid = std::min<uint32_t>((items + RW - 1) / RW, (uint32_t)num_sms * 2);
    return launch_pdl(rows_in_kernel<R>, dim3(grid), dim3(RT), (size_t)(op.w0.n ? op.w0.k : op.gu.k) * 4, st, pdl, op);
}
}  // namespace

cudaError_t launch_rows_in(const RowsIn& op, int num_sms, cudaStream_t st, bool pdl) {
    const uint32_t k = op.w0.n ? op.w0.k : op.gu.k;
    if ((!op.w0.n && !op.gu.n) || k % DENSE_PAD || (op.gu.n && (op.gu.k != k || op.gu.n % 128)) || (size_t)k * 4 > 220 * 1024) return cudaErrorInvalidValue;
    if (op.h_out == op.x) return cudaErrorInvalidValue;   // other CTAs still read x
    return rows_in_r<2>(op, num_sms, st, pdl);
}

cudaError_t launch_rows_out(const RowsOut& op, int num_sms, cudaStream_t st, bool pdl) {
    if (!op.w1.n || op.w1.k % DENSE_PAD || (op.w2.n && (op.w2.n != op.w1.n || op.w2.k % DENSE_PAD))) return cudaErrorInvalidValue;
    if ((size_t)(op.w1.k + (op.w2.n ? op.w2.k : 0)) * 4 > 220 * 1024) return cudaErrorInvalidValue;
    return op.w1.n >= (uint32_t)num_sms * 16 ? rows_out_r<2>(op, num_sms, st, pdl) : rows_out_r<1>(op, num_sms, st, pdl);
}

}  // namespace alice
