// Token mixers of layer-stack models (csrc/delta.cu, csrc/latent.cu, csrc/grouped.cu) and the small per-token kernels around them
// (csrc/stack_ops.cu). Sizes are run-time values; positions come from device memory so that a captured step can be replayed.
#pragma once
#include <cmath>

#include "dense.cuh"

namespace alice {

// ---- stack_ops.cu -------------------------------------------------------------------------------
// x[t] <- (set ? 0 : x[t]) + (emb ? emb[tokens[t]] * scale : 0) + (step ? step : 0); columns [n, ld) are zero there and stay so.
struct EnterArgs {
    const bf16* emb = nullptr;
    const int* tokens = nullptr;
    uint32_t vocab = 0, emb_ld = 0, n = 0, ld = 0;
    float scale = 1.f;
    const float* step = nullptr;
    bool set = false;
    float* x = nullptr;
    void* h = nullptr;                // a copy of the result, rows ld apart
    bool h_bf16 = false;
};
cudaError_t launch_enter(const EnterArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);

constexpr uint32_t MAX_NORM_ROWS = 64;
struct NormArgs {
    const float* x = nullptr;
    uint32_t ldx = 0, n = 0, k = 0;   // true and padded length (a row holds k floats); out rows are k apart, zero beyond n
    int norm = NORM_LAYER;            // NORM_NONE: a plain copy
    const float* w = nullptr;
    float eps = 0.f;
    void* out = nullptr;              // may be null
    bool out_bf16 = false;
    float* x_out = nullptr;           // f32 result, rows ldx apart; may be x
    bool gather = false;              // read rows idx[i] instead of i (at most MAX_NORM_ROWS)
    uint32_t idx[MAX_NORM_ROWS] = {};
};
cudaError_t launch_norm(const NormArgs& a, uint32_t rows, cudaStream_t st, bool pdl);

// ---- delta.cu: delta rule with one decay per key channel ----------------------------------------
struct DeltaShape {
    uint32_t heads, kv_heads, dim, vdim, taps;
    uint32_t dp, vp;                  // dim and vdim padded (dp: 64, 128 or 256; vp: multiple of 32)
    uint32_t off_q, off_k, off_v, off_b, conv_cols;   // columns of the projection output; the convolution covers [0, conv_cols)
};
constexpr uint32_t DELTA_MAX_DIM = 256;
inline uint32_t delta_pad_dim(uint32_t d) { return d <= 64 ? 64 : d <= 128 ? 128 : 256; }
constexpr uint32_t DELTA_BLOCK = 16;      // tokens per block of the recurrence

struct DeltaArgs {
    DeltaShape s;
    const float* y = nullptr;         // projections [t][ldy]: q | k | v | b | ...
    uint32_t ldy = 0;
    const float* conv_w = nullptr;    // [taps][conv_cols]
    float* conv_state = nullptr;      // two of [taps - 1][conv_cols], oldest first: the one of a position's parity holds the inputs before it
    const int* pos = nullptr;
    float* state = nullptr;           // [heads][vp][dp]
    float *qn = nullptr, *kn = nullptr, *v = nullptr, *beta = nullptr;   // prepared inputs of the recurrence
    float *pair_inv = nullptr, *pair_b = nullptr;   // [blocks][heads][DELTA_BLOCK][DELTA_BLOCK]
    const float* g = nullptr;         // decays [t][heads][dp]
    float* o = nullptr;               // [t][heads][vdim]
    const float* gate = nullptr;      // sigmoid already applied, [t][heads * vdim]
    const float* norm_w = nullptr;
    float eps = 0.f;
    void* out = nullptr;              // [t][ldo]
    uint32_t ldo = 0;
    bool out_bf16 = false;
};
// short convolution + silu + unit vectors + step sizes; then the convolution's tail moves into its state
cudaError_t launch_delta_prepare(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
cudaError_t launch_delta_scan(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
cudaError_t launch_delta_out(const DeltaArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
// All of it for one token in one launch, the decay and gate projections included; f32 result.
struct DeltaStepArgs {
    DeltaArgs d;
    DenseMat a2, g2;
    uint32_t off_a = 0, off_g = 0;    // columns of their low-rank inputs in y
    const float *a_log = nullptr, *dt_bias = nullptr;
};
inline bool delta_step_fits(const DeltaStepArgs& a) { return a.d.s.vp <= 256 && a.a2.k + a.g2.k <= 8192; }
cudaError_t launch_delta_step(const DeltaStepArgs& a, cudaStream_t st, bool pdl);

// ---- latent.cu: attention over a cached latent ---------------------------------------------------
struct LatentShape {
    uint32_t heads, dim, rot, rot_dims, vdim, q_rank, kv_rank;
    uint32_t qp, cp, rp;              // padded q_rank, kv_rank (64s) and rot (16s): a cache row is cp + rp wide
    uint32_t off_q, off_kv, off_g;    // columns of the projection output
    float scale;
};
constexpr uint32_t LATENT_MAX_RANK = 1024;

struct LatentArgs {
    LatentShape s;
    const float* y = nullptr;         // projections [t][ldy]: query latent | key latent, rotated key | gate
    uint32_t ldy = 0;
    const float *q_norm = nullptr, *kv_norm = nullptr, *sink = nullptr, *freq = nullptr;
    float eps = 0.f;
    const bf16 *uk = nullptr, *uv = nullptr;   // [heads * dim][cp], [heads * vdim][cp]
    const int* pos = nullptr;
    void* cache = nullptr;            // [max_seq][cp + rp]
    bool cache_bf16 = false;
    void* cqn = nullptr;              // normalised query latent [t][qp]
    bool act_bf16 = false;            // type of cqn and out
    bool append = false;              // launch_latent_absorb also puts the token's row into the cache
    const float* q = nullptr;         // [t][heads * (dim + rot)]
    float* ql = nullptr;              // [t][heads][cp + rp]: queries taken into the latent space, rotated part
    float* part = nullptr;            // [t][splits][heads][cp + 2]
    uint32_t splits = 1;
    float* mix = nullptr;             // [t][heads][cp]: weighted latent
    void* out = nullptr;              // [t][ldo]
    uint32_t ldo = 0;
    // tiled prefill: keys and values of every cached token, made from the latent rows
    const bf16 *k_all = nullptr, *v_all = nullptr;   // [ctx][heads * dim], [ctx][heads * vdim]
    bf16* q_rot = nullptr;                           // [t][heads * (dim + rot)], room for the rotated queries
};
// Whether the tensor-core prefill covers these sizes (others take the latent-space path).
inline bool latent_prefill_fits(const LatentShape& s) {
    return s.dim % 8 == 0 && s.rot % 8 == 0 && s.vdim % 8 == 0 && s.dim + s.rot <= 256 && s.vdim <= 256;
}
cudaError_t launch_latent_prefill(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
cudaError_t launch_latent_norm(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
cudaError_t launch_latent_absorb(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
// scores and weighted sums of queries in the latent space (launch_latent_decode: its tensor-core form, bf16 cache)
bool latent_decode_fits(const LatentShape& s);
cudaError_t launch_latent_decode(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
cudaError_t launch_latent_attn(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
cudaError_t launch_latent_out(const LatentArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);

// ---- grouped.cu: attention whose key / value heads serve groups of query heads ---------------------
struct GroupedShape {
    uint32_t heads, kv_heads, dim, vdim, rot_dims;
    uint32_t dp, vp;                  // dim and vdim padded to 16
    uint32_t off_k, off_v;            // columns of the projection output (queries start at 0)
    float scale, softcap;             // softcap 0: none
    bool unit_qk;                     // rotated queries and keys over their root mean square
    uint32_t group() const { return heads / kv_heads; }
    // A cache row is [key dp | value vp | 8 unused]: eight rows start in different shared-memory banks as they lie.
    __host__ __device__ uint32_t ld() const { return dp + vp + 8; }
};
constexpr uint32_t GROUPED_MAX_DIM = 512, GROUPED_TILE = 16;   // keys are read in whole tiles: planes of the cache hold multiples of it

struct GroupedArgs {
    GroupedShape s;
    const float* y = nullptr;         // projections [t][ldy]: q | k | v
    uint32_t ldy = 0;
    const float *sink = nullptr, *freq = nullptr;   // sink [heads], -inf for none
    float eps = 0.f;
    const int* pos = nullptr;
    void* cache = nullptr;            // [kv_heads][plane_rows][ld]
    uint32_t plane_rows = 0;
    bool cache_bf16 = false;
    void* q = nullptr;                // prepared queries [kv_heads][t][group][dp], of the cache's type
    void* out = nullptr;              // [t][ldo]
    uint32_t ldo = 0;
    bool act_bf16 = false;            // type of out
    bool bounded = false;             // no score exceeds GROUPED_BOUND: exp needs no running maximum
    // grouped_decode.cu
    bool append = false;              // one token: its cache row is made here too
    uint32_t splits = 1;
    float* part = nullptr;            // [t][splits][heads][vp + 4]
    unsigned int* tickets = nullptr;  // [t][kv_heads * groups of 16 heads], zero between launches
    int* status = nullptr;
};
// Rotation and norm of queries and keys; queries to a.q, keys and values into the cache.
cudaError_t launch_grouped_prepare(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
// In f32 arithmetic throughout, prepared queries and cache of either type.
cudaError_t launch_grouped_attn(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
// On the tensor cores, bf16 cache: many tokens (prepared queries), few tokens (queries straight from the projections).
inline bool grouped_tiled_fits(const GroupedShape& s) { return s.dp <= 256 && s.vp <= 256; }
constexpr float GROUPED_BOUND = 60.0f;   // exp of more would leave too little room in f32
// What no score exceeds: unit queries and keys meet in at most dim, and a cap is one.
inline float grouped_bound(const GroupedShape& s) {
    const float unit = s.unit_qk ? 1.01f * std::fabs(s.scale) * s.dim : INFINITY;   // a little more for their rounding
    return s.softcap > 0.0f ? std::fmin(s.softcap, unit) : unit;
}
cudaError_t launch_grouped_prefill(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);
cudaError_t launch_grouped_decode(const GroupedArgs& a, uint32_t tokens, cudaStream_t st, bool pdl);

}  // namespace alice
