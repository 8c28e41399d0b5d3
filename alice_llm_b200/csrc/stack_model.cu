// Layer-stack models behind the alice_model handle (alice_stack_* of include/alice_cuda.h): a list of layers, each with its
// own token mixer and per-pass state, a looped middle part, a 32-bit residual stream.
//
// One token runs on the row kernels (dense_rows.cu) with f32 activations; several tokens run as tiled products
// (dense_gemm.cu) with bfloat16 activations, or f32 ones when the model was created exact.
#include <cmath>
#include <memory>

#include "glue.cuh"
#include "mixers.cuh"
#include "model_base.cuh"

using namespace alice;

namespace {

constexpr uint32_t CHUNK_SMALL = 256, CHUNK = 2048, TRACE_TOKENS = 256;
constexpr uint32_t DECODE_SPLITS = 128;  // most shares of the context one decoded token's attention is cut into
constexpr uint32_t FEW_TOKENS = 4;       // up to here attention runs in its form for single tokens also where the tiled form exists

struct StackModel;

DenseMat mat_of(const alice_weights* w) {
    DenseMat m;
    if (w) { m.w = reinterpret_cast<const bf16*>(w->d.data); m.n = w->d.rows; m.k = w->d.cols; }
    return m;
}

// Buffers of one forward call, shared by all layers.
struct Scratch {
    uint32_t chunk = 0, wp = 0, ldy = 0, ldf = 0, lda = 0;
    float *x = nullptr, *y = nullptr, *r = nullptr;  // stream, projections, a single token's sum ahead of its norm
    void *h = nullptr, *f = nullptr, *a = nullptr;   // activations: f32, or bf16 in tiled products
    // latent
    float *q = nullptr, *ql = nullptr, *part = nullptr, *mix = nullptr;
    void* cqn = nullptr;
    bf16 *k_all = nullptr, *v_all = nullptr, *q_rot = nullptr;   // keys and values of the whole context and rotated queries (tiled prefill)
    unsigned int* tickets = nullptr;                 // grouped attention
    // delta
    float *qn = nullptr, *kn = nullptr, *pair_inv = nullptr, *pair_b = nullptr, *v = nullptr, *beta = nullptr, *g = nullptr, *gate = nullptr, *o = nullptr;
    bf16* low = nullptr;                             // bf16 copy of the low-rank columns
};

// A token mixer: what it computes from the normalised stream, and what it keeps between tokens (one state per pass).
struct Mixer {
    DenseMat in, o;
    virtual ~Mixer() = default;
    // From the projections in s.y to the mixer's heads in s.a; `pass` selects the state.
    virtual int run(StackModel* m, uint32_t tokens, uint32_t pass) = 0;
    virtual int clear(cudaStream_t st) = 0;
    virtual bool recurrent() const = 0;
    // First column of the projections that a tiled product also leaves in bf16 (in.n: none).
    virtual uint32_t low_column() const { return in.n; }
};

struct StackLayer {
    std::unique_ptr<Mixer> mixer;
    DenseMat gu, down;
    uint32_t ff = 0;
    const float *norm = nullptr, *norm2 = nullptr, *ls1 = nullptr, *ls2 = nullptr, *gate_b = nullptr, *up_b = nullptr, *down_b = nullptr;
};

struct StackModel final : alice_model {
    alice_stack_config cfg{};
    std::vector<StackLayer> layers;
    DenseMat embed, out_head;
    const float *final_norm = nullptr, *loop_step = nullptr;
    const float* pending = nullptr;   // weight of a norm that still stands between s.r and the stream (single tokens, norm after the sum)
    Scratch s;
    uint32_t chunk = 0;
    float* trace = nullptr;
    bool tracing = false;
    uint32_t trace_runs = 0, trace_tokens = 0;

    bool exact() const { return cfg.exact != 0; }
    // bf16 activations: several tokens at once, unless everything is to be in 32 bits
    bool tiled_bf16(uint32_t tokens) const { return tokens > 1 && !exact(); }
    uint32_t runs() const { return cfg.num_layers + (cfg.loop_times ? (cfg.loop_times - 1) * (cfg.loop_stop - cfg.loop_start) : 0); }
    uint32_t max_tokens() const override { return tracing ? std::min(chunk, TRACE_TOKENS) : chunk; }
    int enqueue_step(uint32_t n, bool greedy_feed) override;
    int enqueue_rows(uint32_t n, const uint32_t* rows, uint32_t nrows, float* host_logits) override;
    int clear_state() override;
    bool can_return_to(uint32_t p) const override {
        if (p == pos || p == 0) return true;
        for (const auto& l : layers) if (l.mixer->recurrent()) return false;
        return p < pos;
    }

    int body(uint32_t n);
    int layer(uint32_t i, uint32_t n, uint32_t pass) { return cfg.block == ALICE_BLOCK_POST ? layer_post(i, n, pass) : layer_parallel(i, n, pass); }
    int layer_parallel(uint32_t i, uint32_t n, uint32_t pass);
    int layer_post(uint32_t i, uint32_t n, uint32_t pass);
    int settle();
    int norm() const { return cfg.norm == ALICE_NORM_RMS ? NORM_RMS : NORM_LAYER; }
    NormArgs norm_args(const float* w, bool low) const {
        NormArgs na;
        na.x = s.x; na.ldx = s.wp; na.n = cfg.width; na.k = s.wp; na.norm = norm(); na.w = w; na.eps = cfg.eps; na.out = s.h; na.out_bf16 = low;
        return na;
    }
    int head(uint32_t n, const uint32_t* rows, uint32_t nrows, bool argmax);
    int product(GemmOp& op) {
        MCU(launch_dense_gemm(op, e->num_sms, e->status, e->stream, e->pdl));
        return ALICE_OK;
    }
    // out[t] = W a[t] for every token: the row kernel for one token, a tiled product for more (EPI_STORE, f32 result)
    int project(uint32_t n, const void* a, uint32_t lda, const DenseMat& w, float* out, uint32_t ldo, int epi = EPI_STORE, const float* bias = nullptr,
                const float* a_log = nullptr, uint32_t dim = 1) {
        GemmOp op;
        op.tokens = n; op.a = a; op.lda = lda; op.a_bf16 = tiled_bf16(n); op.w = w; op.epi = epi; op.out = out; op.ldo = ldo;
        op.bias = bias; op.a_log = a_log; op.dim = dim;
        return product(op);
    }
};

// ---- mixers ---------------------------------------------------------------------------------------------

struct LatentMixer final : Mixer {
    LatentShape sh{};
    DenseMat uq, uk, uv;
    const float *q_norm = nullptr, *kv_norm = nullptr, *sink = nullptr, *freq = nullptr;
    std::vector<void*> cache;      // per pass, [max_seq][cp + rp]
    size_t cache_bytes = 0;

    bool recurrent() const override { return false; }
    bool tiled(const StackModel* m) const { return !m->exact() && latent_prefill_fits(sh); }
    int clear(cudaStream_t st) override {
        for (void* c : cache) MCU(cudaMemsetAsync(c, 0, cache_bytes, st));
        return ALICE_OK;
    }
    int run(StackModel* m, uint32_t n, uint32_t pass) override {
        Scratch& s = m->s;
        cudaStream_t st = m->e->stream;
        const bool pdl = m->e->pdl;
        LatentArgs a;
        a.s = sh; a.y = s.y; a.ldy = s.ldy; a.q_norm = q_norm; a.kv_norm = kv_norm; a.sink = sink; a.freq = freq; a.eps = m->cfg.eps;
        a.uk = uk.w; a.uv = uv.w; a.pos = m->d_pos; a.cache = cache[pass]; a.cache_bf16 = !m->exact();
        a.cqn = s.cqn; a.act_bf16 = m->tiled_bf16(n); a.q = s.q; a.ql = s.ql; a.part = s.part; a.mix = s.mix; a.out = s.a; a.ldo = o.k;
        // one CTA per SM: shares of the context times groups of 16 heads times tokens
        a.splits = n <= FEW_TOKENS ? std::max<uint32_t>(1, std::min(DECODE_SPLITS, (uint32_t)m->e->num_sms / ((sh.heads + 15) / 16)) / n) : 1;
        if (n == 1) {
            RowsIn in;
            in.x = s.y + sh.off_q; in.n_x = sh.q_rank; in.norm = NORM_RMS; in.norm_w = q_norm; in.eps = m->cfg.eps; in.w0 = uq; in.y0 = s.q;
            MCU(launch_rows_in(in, m->e->num_sms, st, pdl));
            a.append = true;
        } else {
            MCU(launch_latent_norm(a, n, st, pdl));
            const int rc = m->project(n, s.cqn, sh.qp, uq, s.q, uq.n);
            if (rc) return rc;
        }
        if (n > FEW_TOKENS && tiled(m)) {
            const uint32_t ctx = m->pos + n;   // a tiled step is never replayed, so the host's position is the device's
            GemmOp op;
            op.tokens = ctx; op.a = cache[pass]; op.lda = sh.cp + sh.rp; op.a_bf16 = true; op.out_bf16 = true;
            op.w = uk; op.out = s.k_all; op.ldo = uk.n;
            int erc = m->product(op);
            op.w = uv; op.out = s.v_all; op.ldo = uv.n;
            if (!erc) erc = m->product(op);
            if (erc) return erc;
            a.k_all = s.k_all; a.v_all = s.v_all; a.q_rot = s.q_rot;
            MCU(launch_latent_prefill(a, n, st, pdl));
            return ALICE_OK;
        }
        MCU(launch_latent_absorb(a, n, st, pdl));
        MCU(launch_latent_attn(a, n, st, pdl));
        MCU(launch_latent_out(a, n, st, pdl));
        return ALICE_OK;
    }
};

struct DeltaMixer final : Mixer {
    DeltaShape sh{};
    DenseMat a2, g2;
    uint32_t off_a = 0, off_g = 0;
    const float *conv = nullptr, *a_log = nullptr, *dt_bias = nullptr, *norm = nullptr;
    struct State { float *conv, *s; };
    std::vector<State> states;     // per pass
    size_t conv_bytes = 0, state_bytes = 0;

    bool recurrent() const override { return true; }
    uint32_t low_column() const override { return off_a; }
    int clear(cudaStream_t st) override {
        for (const State& p : states) {
            MCU(cudaMemsetAsync(p.conv, 0, conv_bytes, st));
            MCU(cudaMemsetAsync(p.s, 0, state_bytes, st));
        }
        return ALICE_OK;
    }
    int run(StackModel* m, uint32_t n, uint32_t pass) override {
        Scratch& s = m->s;
        cudaStream_t st = m->e->stream;
        const bool pdl = m->e->pdl, low = m->tiled_bf16(n);
        DeltaArgs a;
        a.s = sh; a.y = s.y; a.ldy = s.ldy; a.conv_w = conv; a.conv_state = states[pass].conv; a.state = states[pass].s;
        a.qn = s.qn; a.kn = s.kn; a.pair_inv = s.pair_inv; a.pair_b = s.pair_b; a.v = s.v; a.beta = s.beta; a.g = s.g; a.o = s.o; a.gate = s.gate; a.norm_w = norm; a.eps = m->cfg.eps;
        a.out = s.a; a.ldo = o.k; a.out_bf16 = low; a.pos = m->d_pos;
        DeltaStepArgs sa;
        sa.d = a; sa.a2 = a2; sa.g2 = g2; sa.off_a = off_a; sa.off_g = off_g; sa.a_log = a_log; sa.dt_bias = dt_bias;
        if (n == 1 && delta_step_fits(sa)) {
            MCU(launch_delta_step(sa, st, pdl));
            return ALICE_OK;
        }
        const uint32_t ldl = in.n - off_a;
        const void* va = low ? (const void*)s.low : (const void*)(s.y + off_a);
        const void* vg = low ? (const void*)(s.low + (off_g - off_a)) : (const void*)(s.y + off_g);
        const uint32_t ld = low ? ldl : s.ldy;
        int rc = m->project(n, va, ld, a2, s.g, a2.n, EPI_DECAY, dt_bias, a_log, sh.dp);
        if (!rc) rc = m->project(n, vg, ld, g2, s.gate, g2.n, EPI_SIGMOID);
        if (rc) return rc;
        MCU(launch_delta_prepare(a, n, st, pdl));
        MCU(launch_delta_scan(a, n, st, pdl));
        MCU(launch_delta_out(a, n, st, pdl));
        return ALICE_OK;
    }
};

struct GroupedMixer final : Mixer {
    GroupedShape sh{};
    const float *sink = nullptr, *freq = nullptr;
    std::vector<void*> cache;      // per pass, [kv_heads][plane_rows][ld]
    uint32_t plane_rows = 0;
    size_t cache_bytes = 0;

    bool recurrent() const override { return false; }
    bool tiled(const StackModel* m) const { return !m->exact() && grouped_tiled_fits(sh); }
    uint32_t head_groups() const { return sh.kv_heads * ((sh.group() + 15) / 16); }   // CTAs of a share of the context
    int clear(cudaStream_t st) override {
        for (void* c : cache) MCU(cudaMemsetAsync(c, 0, cache_bytes, st));
        return ALICE_OK;
    }
    int run(StackModel* m, uint32_t n, uint32_t pass) override {
        Scratch& s = m->s;
        cudaStream_t st = m->e->stream;
        const bool pdl = m->e->pdl;
        GroupedArgs a;
        a.s = sh; a.y = s.y; a.ldy = s.ldy; a.sink = sink; a.freq = freq; a.eps = m->cfg.eps; a.pos = m->d_pos; a.cache = cache[pass]; a.plane_rows = plane_rows;
        a.cache_bf16 = !m->exact(); a.q = m->exact() ? (void*)s.q : (void*)s.q_rot; a.out = s.a; a.ldo = o.k; a.act_bf16 = m->tiled_bf16(n);
        a.bounded = grouped_bound(sh) <= GROUPED_BOUND; a.part = s.part; a.tickets = s.tickets; a.status = m->e->status;
        const bool few = n <= FEW_TOKENS && tiled(m);
        a.append = few && n == 1;
        if (!a.append) MCU(launch_grouped_prepare(a, n, st, pdl));
        if (few) {
            // one CTA per SM: shares of the context times heads times tokens
            a.splits = std::max<uint32_t>(1, std::min(DECODE_SPLITS, (uint32_t)m->e->num_sms / head_groups()) / n);
            MCU(launch_grouped_decode(a, n, st, pdl));
        } else if (tiled(m)) {
            MCU(launch_grouped_prefill(a, n, st, pdl));
        } else {
            MCU(launch_grouped_attn(a, n, st, pdl));
        }
        return ALICE_OK;
    }
};

// ---- the step -------------------------------------------------------------------------------------------

// x + ls1 * mixer(h) + ls2 * mlp(h), both of the same normalised stream.
int StackModel::layer_parallel(uint32_t i, uint32_t n, uint32_t pass) {
    StackLayer& L = layers[i];
    Mixer& mx = *L.mixer;
    cudaStream_t st = e->stream;
    const bool low = tiled_bf16(n);
    if (n == 1) {
        RowsIn in;
        in.x = s.x; in.n_x = cfg.width; in.norm = norm(); in.norm_w = L.norm; in.eps = cfg.eps;
        in.w0 = mx.in; in.y0 = s.y;
        if (L.ff) { in.gu = L.gu; in.gate_b = L.gate_b; in.up_b = L.up_b; in.y1 = static_cast<float*>(s.f); }
        MCU(launch_rows_in(in, e->num_sms, st, e->pdl));
        const int rc = mx.run(this, n, pass);
        if (rc) return rc;
        RowsOut out;
        out.w1 = mx.o; out.a = static_cast<const float*>(s.a); out.s1 = L.ls1; out.x = out.out = s.x;
        if (L.ff) { out.w2 = L.down; out.f = static_cast<const float*>(s.f); out.s2 = L.ls2; out.b2 = L.down_b; }
        MCU(launch_rows_out(out, e->num_sms, st, e->pdl));
        return ALICE_OK;
    }
    MCU(launch_norm(norm_args(L.norm, low), n, st, e->pdl));
    int rc;
    {
        GemmOp op;
        op.tokens = n; op.a = s.h; op.lda = s.wp; op.a_bf16 = low; op.w = mx.in; op.out = s.y; op.ldo = s.ldy;
        if (low && mx.low_column() < mx.in.n) { op.out2 = s.low; op.col2 = mx.low_column(); op.ld2 = mx.in.n - op.col2; }
        if ((rc = product(op))) return rc;
    }
    if (L.ff) {
        GemmOp op;
        op.tokens = n; op.a = s.h; op.lda = s.wp; op.a_bf16 = low; op.w = L.gu; op.epi = EPI_SWIGLU; op.out = s.f; op.ldo = L.down.k; op.out_bf16 = low;
        op.bias = L.gate_b; op.bias2 = L.up_b;
        if ((rc = product(op))) return rc;
    }
    if ((rc = mx.run(this, n, pass))) return rc;
    GemmOp op;
    op.tokens = n; op.a = s.a; op.lda = mx.o.k; op.a_bf16 = low; op.w = mx.o; op.epi = EPI_RESID; op.out = s.x; op.ldo = s.wp; op.scale = L.ls1;
    if ((rc = product(op))) return rc;
    if (L.ff) {
        op.a = s.f; op.lda = L.down.k; op.w = L.down; op.scale = L.ls2; op.bias = L.down_b;
        if ((rc = product(op))) return rc;
    }
    return ALICE_OK;
}

// x <- norm1(alpha * x + mixer(x)), x <- norm2(alpha * x + mlp(x)). A single token's sum stays in s.r until the next product
// takes its norm on the way in and leaves the stream in s.x; of several tokens the stream is also kept in s.h as the products read it.
int StackModel::layer_post(uint32_t i, uint32_t n, uint32_t pass) {
    StackLayer& L = layers[i];
    Mixer& mx = *L.mixer;
    cudaStream_t st = e->stream;
    const bool low = tiled_bf16(n);
    int rc;
    if (n == 1) {
        RowsIn in;
        in.n_x = cfg.width; in.eps = cfg.eps;
        in.x = pending ? s.r : s.x; in.norm = pending ? norm() : NORM_NONE; in.norm_w = pending; in.h_out = pending ? s.x : nullptr;
        in.w0 = mx.in; in.y0 = s.y;
        MCU(launch_rows_in(in, e->num_sms, st, e->pdl));
        if ((rc = mx.run(this, n, pass))) return rc;
        RowsOut out;
        out.w1 = mx.o; out.a = static_cast<const float*>(s.a); out.alpha = cfg.alpha; out.x = s.x; out.out = s.r;
        MCU(launch_rows_out(out, e->num_sms, st, e->pdl));
        pending = L.norm;
        if (!L.ff) return ALICE_OK;
        in = RowsIn();
        in.n_x = cfg.width; in.eps = cfg.eps; in.x = s.r; in.norm = norm(); in.norm_w = pending; in.h_out = s.x;
        in.gu = L.gu; in.gate_b = L.gate_b; in.up_b = L.up_b; in.y1 = static_cast<float*>(s.f);
        MCU(launch_rows_in(in, e->num_sms, st, e->pdl));
        out.w1 = L.down; out.a = static_cast<const float*>(s.f);
        MCU(launch_rows_out(out, e->num_sms, st, e->pdl));
        pending = L.norm2;
        return ALICE_OK;
    }
    GemmOp op;
    op.tokens = n; op.a = s.h; op.lda = s.wp; op.a_bf16 = low; op.w = mx.in; op.out = s.y; op.ldo = s.ldy;
    if (low && mx.low_column() < mx.in.n) { op.out2 = s.low; op.col2 = mx.low_column(); op.ld2 = mx.in.n - op.col2; }
    if ((rc = product(op))) return rc;
    if ((rc = mx.run(this, n, pass))) return rc;
    auto join = [&](const void* a, const DenseMat& w, const float* norm_w) -> int {
        GemmOp op;
        op.tokens = n; op.a = a; op.lda = w.k; op.a_bf16 = low; op.w = w; op.epi = EPI_RESID; op.out = s.x; op.ldo = s.wp; op.alpha = cfg.alpha;
        const int rc = product(op);
        if (rc) return rc;
        NormArgs na = norm_args(norm_w, low);
        na.x_out = s.x;
        MCU(launch_norm(na, n, st, e->pdl));
        return ALICE_OK;
    };
    if ((rc = join(s.a, mx.o, L.norm)) || !L.ff) return rc;
    op = GemmOp();
    op.tokens = n; op.a = s.h; op.lda = s.wp; op.a_bf16 = low; op.w = L.gu; op.epi = EPI_SWIGLU; op.out = s.f; op.ldo = L.down.k; op.out_bf16 = low;
    op.bias = L.gate_b; op.bias2 = L.up_b;
    if ((rc = product(op))) return rc;
    return join(s.f, L.down, L.norm2);
}

// The stream in s.x, whatever norm still stands before it.
int StackModel::settle() {
    if (!pending) return ALICE_OK;
    NormArgs na = norm_args(pending, false);
    na.x = s.r; na.x_out = s.x; na.out = nullptr;
    MCU(launch_norm(na, 1, e->stream, e->pdl));
    pending = nullptr;
    return ALICE_OK;
}

int StackModel::body(uint32_t n) {
    cudaStream_t st = e->stream;
    EnterArgs ea;
    ea.emb = embed.w; ea.tokens = d_token; ea.vocab = vocab; ea.emb_ld = embed.k; ea.n = cfg.width; ea.ld = s.wp; ea.scale = cfg.embed_scale;
    ea.set = true; ea.x = s.x;
    if (cfg.block == ALICE_BLOCK_POST && n > 1) { ea.h = s.h; ea.h_bf16 = tiled_bf16(n); }   // layers read the stream itself: its copy as the products take it
    MCU(launch_enter(ea, n, st, e->pdl));
    pending = nullptr;
    int rc;
    trace_runs = 0; trace_tokens = n;
    auto one = [&](uint32_t i, uint32_t pass) -> int {
        int rc = layer(i, n, pass);
        if (rc) return rc;
        if (tracing) {
            if ((rc = settle())) return rc;
            MCU(cudaMemcpy2DAsync(trace + (size_t)trace_runs * n * cfg.width, (size_t)cfg.width * 4, s.x, (size_t)s.wp * 4, (size_t)cfg.width * 4, n,
                                  cudaMemcpyDeviceToDevice, st));
            trace_runs++;
        }
        return ALICE_OK;
    };
    const uint32_t a = cfg.loop_times ? cfg.loop_start : cfg.num_layers, b = cfg.loop_times ? cfg.loop_stop : cfg.num_layers;
    for (uint32_t i = 0; i < a; i++) if ((rc = one(i, 0))) return rc;
    for (uint32_t t = 0; t < cfg.loop_times; t++) {
        EnterArgs la = ea;
        la.set = false;
        if (t == 0) la.emb = nullptr;
        la.step = loop_step + (size_t)t * cfg.width;
        if ((rc = settle())) return rc;
        if (b > a) MCU(launch_enter(la, n, st, e->pdl));
        for (uint32_t i = a; i < b; i++) if ((rc = one(i, t))) return rc;
    }
    for (uint32_t i = b; i < cfg.num_layers; i++) if ((rc = one(i, 0))) return rc;
    return settle();
}

// Logits of the given rows of the stream (at most MAX_NORM_ROWS).
int StackModel::head(uint32_t n, const uint32_t* rows, uint32_t nrows, bool argmax) {
    if (nrows == 1) {
        RowsIn in;
        in.x = s.x + (size_t)rows[0] * s.wp; in.n_x = cfg.width; in.norm = norm(); in.norm_w = final_norm; in.eps = cfg.eps;
        in.w0 = out_head; in.y0 = logits;
        if (argmax) in.argmax_key = argmax_keys;
        MCU(launch_rows_in(in, e->num_sms, e->stream, e->pdl));
        return ALICE_OK;
    }
    const bool low = tiled_bf16(n);
    NormArgs na = norm_args(final_norm, low);
    na.gather = true;
    for (uint32_t i = 0; i < nrows; i++) na.idx[i] = rows[i];
    MCU(launch_norm(na, nrows, e->stream, e->pdl));
    GemmOp op;
    op.tokens = nrows; op.a = s.h; op.lda = s.wp; op.a_bf16 = low; op.w = out_head; op.out = logits; op.ldo = vocab;
    return product(op);
}

int StackModel::enqueue_step(uint32_t n, bool greedy_feed) {
    int rc = body(n);
    const uint32_t last = n - 1;
    if (!rc) rc = head(n, &last, 1, greedy_feed);
    if (rc) return rc;
    MCU(launch_finish_step(argmax_keys, 1, d_token, d_pos, d_trace, greedy_feed ? 1 : 0, n, nullptr, e->stream, e->pdl));
    return ALICE_OK;
}

int StackModel::enqueue_rows(uint32_t n, const uint32_t* rows, uint32_t nrows, float* host_logits) {
    int rc = body(n);
    for (uint32_t i = 0; i < nrows && !rc; i += MAX_NORM_ROWS) {
        const uint32_t k = std::min(MAX_NORM_ROWS, nrows - i);
        rc = head(n, rows + i, k, false);
        if (!rc) MCU(cudaMemcpyAsync(host_logits + (size_t)i * vocab, logits, (size_t)k * vocab * 4, cudaMemcpyDeviceToHost, e->stream));
    }
    if (rc) return rc;
    MCU(launch_finish_step(argmax_keys, 1, d_token, d_pos, d_trace, 0, n, nullptr, e->stream, e->pdl));
    return ALICE_OK;
}

int StackModel::clear_state() {
    for (auto& l : layers) {
        const int rc = l.mixer->clear(e->stream);
        if (rc) return rc;
    }
    return ALICE_OK;
}

// ---- creation -------------------------------------------------------------------------------------------

struct Builder {
    StackModel* m;
    const char* who = "alice_stack_create";
    int rc = ALICE_OK;

    const float* floats(const float* host, size_t n, const char* name) {
        if (rc) return nullptr;
        if (!host) { rc = alice_fail(ALICE_E_INVALID, "%s: %s is null", who, name); return nullptr; }
        float* d = nullptr;
        rc = dev_alloc(m, &d, n);
        if (rc) return nullptr;
        const cudaError_t err = cudaMemcpy(d, host, n * sizeof(float), cudaMemcpyHostToDevice);
        if (err != cudaSuccess) rc = alice_cuda_fail(err, who);
        return d;
    }
    template <class T>
    T* zeros(size_t n) {
        T* d = nullptr;
        if (!rc) rc = dev_alloc(m, &d, n);
        if (!rc) {
            const cudaError_t err = cudaMemset(d, 0, std::max<size_t>(n, 1) * sizeof(T));
            if (err != cudaSuccess) rc = alice_cuda_fail(err, who);
        }
        return d;
    }
    DenseMat matrix(const alice_weights* w, uint32_t rows, uint32_t cols, const char* name) {
        if (rc) return {};
        if (!w || w->d.fmt != WF_BF16 || w->d.rows != rows || w->d.cols != cols || ((uintptr_t)w->d.data & 15)) {
            rc = alice_fail(w ? ALICE_E_SHAPE : ALICE_E_INVALID, "%s: %s must be bf16 [%u x %u] (is %u x %u)", who, name, rows, cols, w ? w->d.rows : 0, w ? w->d.cols : 0);
            return {};
        }
        return mat_of(w);
    }
    void shape(const char* what) { if (!rc) rc = alice_fail(ALICE_E_SHAPE, "%s: %s", who, what); }
};

uint32_t P(uint32_t v) { return pad_to(v, DENSE_PAD); }

// Frequencies of the rotated pairs, in double and rounded once. With a factor, wavelengths above original / low turn that much
// slower, those below original / high stay, and between the two the share of the original grows linearly.
const float* rotation(Builder& b, const alice_stack_layer& L) {
    std::vector<float> f(std::max<uint32_t>(1, L.rot_dims / 2));
    for (uint32_t i = 0; i < L.rot_dims / 2; i++) {
        double x = std::pow(L.rot_base, -2.0 * i / L.rot_dims);
        if (L.rot_factor != 0.0) {
            const double wave = 2.0 * 3.14159265358979323846 / x;
            if (wave > L.rot_original / L.rot_low) {
                x /= L.rot_factor;
            } else if (wave >= L.rot_original / L.rot_high && L.rot_high > L.rot_low) {
                const double keep = (L.rot_original / wave - L.rot_low) / (L.rot_high - L.rot_low);
                x = (1.0 - keep) * x / L.rot_factor + keep * x;
            }
        }
        f[i] = (float)x;
    }
    return b.floats(f.data(), f.size(), "freq");
}

void build_latent(Builder& b, const alice_stack_layer& L, uint32_t wp, uint32_t passes, LatentMixer& mx) {
    StackModel* m = b.m;
    LatentShape& s = mx.sh;
    if (!L.heads || !L.dim || !L.vdim || !L.q_rank || !L.kv_rank) return b.shape("latent mixer with a zero size");
    if (L.rot_dims % 2 || L.rot_dims > L.rot_dim) return b.shape("rotated dimensions must be even and lie within rot_dim");
    if (L.kv_rank > LATENT_MAX_RANK) return b.shape("kv_rank above 1024");
    s.heads = L.heads; s.dim = L.dim; s.rot = L.rot_dim; s.rot_dims = L.rot_dims; s.vdim = L.vdim; s.q_rank = L.q_rank; s.kv_rank = L.kv_rank;
    s.qp = P(L.q_rank); s.cp = P(L.kv_rank); s.rp = pad_to(L.rot_dim, 16); s.scale = L.scale;
    s.off_q = 0; s.off_kv = s.qp; s.off_g = s.off_kv + P(L.kv_rank + L.rot_dim);
    mx.in = b.matrix(L.in, s.off_g + P(L.heads * L.vdim), wp, "in");
    mx.uq = b.matrix(L.uq, L.heads * (L.dim + L.rot_dim), s.qp, "uq");
    mx.uk = b.matrix(L.uk, L.heads * L.dim, s.cp, "uk");
    mx.uv = b.matrix(L.uv, L.heads * L.vdim, s.cp, "uv");
    mx.o = b.matrix(L.o, m->cfg.width, P(L.heads * L.vdim), "o");
    mx.q_norm = b.floats(L.q_norm, L.q_rank, "q_norm");
    mx.kv_norm = b.floats(L.kv_norm, L.kv_rank, "kv_norm");
    mx.sink = b.floats(L.sink, L.heads, "sink");
    mx.freq = rotation(b, L);
    mx.cache_bytes = (size_t)m->max_seq * (s.cp + s.rp) * (m->exact() ? 4 : 2);
    for (uint32_t p = 0; p < passes; p++) mx.cache.push_back(b.zeros<uint8_t>(mx.cache_bytes));
}

void build_delta(Builder& b, const alice_stack_layer& L, uint32_t wp, uint32_t passes, DeltaMixer& mx) {
    DeltaShape& s = mx.sh;
    if (!L.heads || !L.kv_heads || L.heads % L.kv_heads || !L.dim || !L.vdim || !L.conv_taps || !L.decay_rank || !L.gate_rank)
        return b.shape("delta mixer with a zero size, or heads no multiple of kv_heads");
    if (L.dim > DELTA_MAX_DIM) return b.shape("delta mixer with more than 256 key channels");
    s.heads = L.heads; s.kv_heads = L.kv_heads; s.dim = L.dim; s.vdim = L.vdim; s.taps = L.conv_taps;
    s.dp = delta_pad_dim(L.dim); s.vp = pad_to(L.vdim, 32);
    s.off_q = 0; s.off_k = P(L.kv_heads * L.dim); s.off_v = 2 * s.off_k; s.off_b = s.conv_cols = s.off_v + P(L.heads * L.vdim);
    mx.off_a = s.off_b + P(L.heads); mx.off_g = mx.off_a + P(L.decay_rank);
    mx.in = b.matrix(L.in, mx.off_g + P(L.gate_rank), wp, "in");
    mx.a2 = b.matrix(L.a2, L.heads * s.dp, P(L.decay_rank), "a2");
    mx.g2 = b.matrix(L.g2, L.heads * L.vdim, P(L.gate_rank), "g2");
    mx.o = b.matrix(L.o, b.m->cfg.width, P(L.heads * L.vdim), "o");
    mx.conv = b.floats(L.conv, (size_t)s.conv_cols * L.conv_taps, "conv");
    mx.a_log = b.floats(L.a_log, L.heads, "a_log");
    mx.dt_bias = b.floats(L.dt_bias, (size_t)L.heads * s.dp, "dt_bias");
    mx.norm = b.floats(L.head_norm, L.vdim, "head_norm");
    mx.conv_bytes = (size_t)2 * std::max<uint32_t>(1, L.conv_taps - 1) * s.conv_cols * 4;
    mx.state_bytes = (size_t)L.heads * s.vp * s.dp * 4;
    for (uint32_t p = 0; p < passes; p++) {
        DeltaMixer::State st{b.zeros<float>(mx.conv_bytes / 4), b.zeros<float>(mx.state_bytes / 4)};
        mx.states.push_back(st);
    }
}

void build_grouped(Builder& b, const alice_stack_layer& L, uint32_t wp, uint32_t passes, GroupedMixer& mx) {
    StackModel* m = b.m;
    GroupedShape& s = mx.sh;
    if (!L.heads || !L.kv_heads || L.heads % L.kv_heads || !L.dim || !L.vdim) return b.shape("grouped mixer with a zero size, or heads no multiple of kv_heads");
    if (L.rot_dims % 2 || L.rot_dims > L.dim) return b.shape("rotated dimensions must be even and lie within dim");
    if (L.dim > GROUPED_MAX_DIM || L.vdim > GROUPED_MAX_DIM) return b.shape("grouped mixer with more than 512 dimensions a head");
    if (L.softcap < 0.0f) return b.shape("negative softcap");
    s.heads = L.heads; s.kv_heads = L.kv_heads; s.dim = L.dim; s.vdim = L.vdim; s.rot_dims = L.rot_dims; s.dp = pad_to(L.dim, 16); s.vp = pad_to(L.vdim, 16);
    s.off_k = P(L.heads * L.dim); s.off_v = s.off_k + P(L.kv_heads * L.dim); s.scale = L.scale; s.softcap = L.softcap; s.unit_qk = L.unit_qk != 0;
    mx.in = b.matrix(L.in, s.off_v + P(L.kv_heads * L.vdim), wp, "in");
    mx.o = b.matrix(L.o, m->cfg.width, P(L.heads * L.vdim), "o");
    const std::vector<float> none(L.heads, -INFINITY);
    mx.sink = b.floats(L.sink ? L.sink : none.data(), L.heads, "sink");
    mx.freq = rotation(b, L);
    mx.plane_rows = pad_to(m->max_seq, 64);
    static_assert(64 % GROUPED_TILE == 0, "whole tiles in a plane");
    mx.cache_bytes = (size_t)L.kv_heads * mx.plane_rows * s.ld() * (m->exact() ? 4 : 2);
    for (uint32_t p = 0; p < passes; p++) mx.cache.push_back(b.zeros<uint8_t>(mx.cache_bytes));
}

// Scratch for the largest layer of each kind.
void build_scratch(Builder& b) {
    StackModel* m = b.m;
    Scratch& s = m->s;
    // where attention of many tokens runs in the latent space, fewer of them go at once
    bool small = m->exact();
    for (const auto& L : m->layers)
        if (const auto* x = dynamic_cast<const LatentMixer*>(L.mixer.get())) small |= !x->tiled(m);
    m->chunk = std::min<uint32_t>(small ? CHUNK_SMALL : CHUNK, pad_to(m->max_seq, 64));
    const uint32_t M = m->chunk, ML = small ? M : std::min(M, FEW_TOKENS);
    uint32_t k_all = 0, v_all = 0, q_rot = 0, few = 0, tickets = 0;   // few: partial sums of a share, for FEW_TOKENS at once
    uint32_t ldy = 0, ldf = 0, lda = 0, q = 0, ql = 0, part = 0, mix = 0, qp = 0, kd = 0, v = 0, h = 0, g = 0, o = 0, low = 0;
    for (const auto& L : m->layers) {
        ldy = std::max(ldy, L.mixer->in.n);
        lda = std::max(lda, L.mixer->o.k);
        ldf = std::max(ldf, L.down.k);
        if (const auto* x = dynamic_cast<const LatentMixer*>(L.mixer.get())) {
            const LatentShape& z = x->sh;
            if (x->tiled(m)) { k_all = std::max(k_all, x->uk.n); v_all = std::max(v_all, x->uv.n); q_rot = std::max(q_rot, x->uq.n); }
            q = std::max(q, x->uq.n); qp = std::max(qp, z.qp);
            ql = std::max(ql, z.heads * (z.cp + z.rp)); part = std::max(part, z.heads * (z.cp + 2)); mix = std::max(mix, z.heads * z.cp);
        } else if (const auto* x = dynamic_cast<const GroupedMixer*>(L.mixer.get())) {
            const GroupedShape& z = x->sh;
            (m->exact() ? q : q_rot) = std::max(m->exact() ? q : q_rot, z.heads * z.dp);
            if (x->tiled(m)) { few = std::max(few, z.heads * (z.vp + 4)); tickets = std::max(tickets, FEW_TOKENS * x->head_groups()); }
        } else if (const auto* x = dynamic_cast<const DeltaMixer*>(L.mixer.get())) {
            const DeltaShape& z = x->sh;
            kd = std::max(kd, z.kv_heads * z.dp); v = std::max(v, z.heads * z.vp); h = std::max(h, z.heads);
            g = std::max(g, z.heads * z.dp); o = std::max(o, z.heads * z.vdim); low = std::max(low, x->in.n - x->off_a);
        }
    }
    s.chunk = M; s.wp = P(m->cfg.width); s.ldy = ldy;
    s.x = b.zeros<float>((size_t)M * s.wp);
    s.y = b.zeros<float>((size_t)M * ldy);
    s.r = b.zeros<float>(s.wp);
    s.h = b.zeros<float>((size_t)M * s.wp);
    s.f = b.zeros<float>((size_t)M * ldf);
    s.a = b.zeros<float>((size_t)M * lda);     // heads * vdim columns and the padding of each mixer's own stride
    s.q = b.zeros<float>((size_t)M * q);
    s.cqn = b.zeros<float>((size_t)M * qp);
    s.ql = b.zeros<float>((size_t)ML * ql);
    s.part = b.zeros<float>(std::max((size_t)std::max(ML, DECODE_SPLITS) * part, (size_t)std::max(FEW_TOKENS, DECODE_SPLITS) * few));
    s.tickets = b.zeros<unsigned int>(tickets);
    s.mix = b.zeros<float>((size_t)ML * mix);
    s.k_all = b.zeros<bf16>((size_t)m->max_seq * k_all);
    s.q_rot = b.zeros<bf16>((size_t)M * q_rot);
    s.v_all = b.zeros<bf16>((size_t)m->max_seq * v_all);
    s.qn = b.zeros<float>((size_t)M * kd); s.kn = b.zeros<float>((size_t)M * kd);
    s.pair_inv = b.zeros<float>((size_t)M * h * DELTA_BLOCK); s.pair_b = b.zeros<float>((size_t)M * h * DELTA_BLOCK);
    s.v = b.zeros<float>((size_t)M * v); s.beta = b.zeros<float>((size_t)M * h); s.g = b.zeros<float>((size_t)M * g);
    s.gate = b.zeros<float>((size_t)M * o); s.o = b.zeros<float>((size_t)M * o);
    s.low = b.zeros<bf16>((size_t)M * low);
    m->logits = b.zeros<float>((size_t)MAX_NORM_ROWS * m->vocab);
    m->argmax_keys = b.zeros<unsigned long long>(1);
    m->d_pos = b.zeros<int>(1);
    m->d_token = b.zeros<int>(M);
    m->d_trace = b.zeros<int>(m->max_seq);
}

}  // namespace

extern "C" {

int32_t alice_stack_create(alice_engine* e, const alice_stack_config* cfg, const alice_stack_layer* layers, const alice_weights* embed,
                           const float* final_norm, alice_model** out) {
    const char* who = "alice_stack_create";
    if (!e || !cfg || !layers || !embed || !final_norm || !out) return alice_fail(ALICE_E_INVALID, "%s: null argument", who);
    *out = nullptr;
    const alice_stack_config& c = *cfg;
    if (!c.num_layers || !c.width || !c.vocab_size || !c.max_seq_len) return alice_fail(ALICE_E_SHAPE, "%s: zero dimension in config", who);
    if (c.loop_times && (c.loop_start > c.loop_stop || c.loop_stop > c.num_layers || !c.loop_step))
        return alice_fail(ALICE_E_SHAPE, "%s: loop %u .. %u of %u layers", who, c.loop_start, c.loop_stop, c.num_layers);
    if (c.block > ALICE_BLOCK_POST || c.norm > ALICE_NORM_RMS) return alice_fail(ALICE_E_UNSUPPORTED, "%s: block %u, norm %u", who, c.block, c.norm);
    if (e->tp_world > 1) return alice_fail(ALICE_E_UNSUPPORTED, "%s: layer-stack models run on one GPU", who);
    MCU(cudaSetDevice(e->device));
    auto* m = new StackModel();
    m->e = e; m->cfg = c; m->vocab = c.vocab_size; m->max_seq = c.max_seq_len;
    alice_engine_retain(e);
    Builder b{m};
    const uint32_t wp = P(c.width);
    m->embed = b.matrix(embed, c.vocab_size, wp, "embed");
    m->out_head = c.head ? b.matrix(c.head, c.vocab_size, wp, "head") : m->embed;
    m->final_norm = b.floats(final_norm, c.width, "final_norm");
    if (c.loop_times) m->loop_step = b.floats(c.loop_step, (size_t)c.loop_times * c.width, "loop_step");
    for (uint32_t i = 0; i < c.num_layers && !b.rc; i++) {
        const alice_stack_layer& L = layers[i];
        const uint32_t passes = c.loop_times && i >= c.loop_start && i < c.loop_stop ? c.loop_times : 1;
        StackLayer sl;
        if (L.mixer == ALICE_MIX_LATENT) {
            auto mx = std::make_unique<LatentMixer>();
            build_latent(b, L, wp, passes, *mx);
            sl.mixer = std::move(mx);
        } else if (L.mixer == ALICE_MIX_DELTA) {
            auto mx = std::make_unique<DeltaMixer>();
            build_delta(b, L, wp, passes, *mx);
            sl.mixer = std::move(mx);
        } else if (L.mixer == ALICE_MIX_GROUPED) {
            auto mx = std::make_unique<GroupedMixer>();
            build_grouped(b, L, wp, passes, *mx);
            sl.mixer = std::move(mx);
        } else {
            b.rc = alice_fail(ALICE_E_UNSUPPORTED, "%s: layer %u has an unknown mixer %u", who, i, L.mixer);
            break;
        }
        sl.norm = b.floats(L.norm, c.width, "norm");
        const bool post = c.block == ALICE_BLOCK_POST;
        auto optional = [&](const float* p, size_t n, const char* name) { return p ? b.floats(p, n, name) : nullptr; };
        if (!post) sl.ls1 = b.floats(L.ls1, c.width, "ls1");
        if (L.ff) {
            sl.ff = L.ff;
            sl.gu = b.matrix(L.gu, 2 * P(L.ff), wp, "gu");
            sl.down = b.matrix(L.down, c.width, P(L.ff), "down");
            if (post) sl.norm2 = b.floats(L.norm2, c.width, "norm2");
            else sl.ls2 = b.floats(L.ls2, c.width, "ls2");
            if (post && L.down_bias) b.shape("a bias on the way out of a feed-forward whose norm comes behind the sum");
            if (!L.gate_bias != !L.up_bias) b.shape("gate and up biases come together");
            sl.gate_b = optional(L.gate_bias, P(L.ff), "gate_bias");
            sl.up_b = optional(L.up_bias, P(L.ff), "up_bias");
            if (!post) sl.down_b = b.floats(L.down_bias, c.width, "down_bias");
        }
        m->layers.push_back(std::move(sl));
    }
    if (!b.rc) build_scratch(b);
    if (!b.rc && cudaDeviceSynchronize() != cudaSuccess) b.rc = alice_cuda_fail(cudaGetLastError(), who);
    if (b.rc) { alice_model_destroy(m); return b.rc; }
    *out = m;
    return ALICE_OK;
}

int32_t alice_stack_trace(alice_model* base, int32_t on) {
    auto* m = dynamic_cast<StackModel*>(base);
    if (!m) return alice_fail(ALICE_E_INVALID, "alice_stack_trace: not a layer-stack model");
    MCU(cudaSetDevice(m->e->device));
    if (on && !m->trace) {
        const int rc = dev_alloc(m, &m->trace, (size_t)m->runs() * TRACE_TOKENS * m->cfg.width);
        if (rc) return rc;
    }
    m->tracing = on != 0;
    return ALICE_OK;
}

int32_t alice_stack_read_trace(alice_model* base, float* out, size_t out_floats, uint32_t* runs, uint32_t* tokens) {
    auto* m = dynamic_cast<StackModel*>(base);
    if (!m || !runs || !tokens) return alice_fail(ALICE_E_INVALID, "alice_stack_read_trace: null argument or not a layer-stack model");
    *runs = m->trace_runs; *tokens = m->trace_tokens;
    if (!out) return ALICE_OK;
    const size_t n = (size_t)m->trace_runs * m->trace_tokens * m->cfg.width;
    if (out_floats < n) return alice_fail(ALICE_E_SHAPE, "alice_stack_read_trace: %zu floats, need %zu", out_floats, n);
    MCU(cudaMemcpyAsync(out, m->trace, n * 4, cudaMemcpyDeviceToHost, m->e->stream));
    MCU(cudaStreamSynchronize(m->e->stream));
    return ALICE_OK;
}

}  // extern "C"
