// The Fuposun design: a pre-norm decoder without positions whose layers differ one by one,
//     x <- x + m * mixer(n1(x)),     x <- x + m * ff(n2(x)),
// with a norm behind the embedding and a soft cap on the logits.  Mixers: attention over latents in a sliding window with
// a gate per head ("latent_attention"), and gated linear attention ("gla").  Feed-forward: dense, a mixture of experts with
// a shared one, or none.  The residual stream is float.
//
// What a sequence keeps: per attention layer a ring of latents as long as the window, per recurrent layer a float state.
// Neither grows with its length.
//
// Steps of a layer.  Everything a mixer takes from its normed input is one matrix; the factor m goes into the epilogue of
// the projection that adds to the stream; the experts' outputs are added in the pass that makes the next norm.
//   latent attention   [dq | dkv | gate] -> norms, latents stored -> queries, then
//     up to 64 tokens (and every pass in float32): queries into latent space (per-head projection) -> attention over the
//       latents -> values out of latent space (per-head projection);
//     more: keys and values of the pass's tokens and of the window in front of them, formed once -> attention on them;
//     -> output projection
//   gla                [q | k | v | gate | low-rank decay] -> recurrence with norm and gate -> output projection
//   dense              silu(gate) * up -> down
//   experts            router -> choice and places -> gate/up and down as projections in row groups; the shared expert is
//                      added to the stream directly
//
// Sizes that the kernels do not take as they are get padded in memory with zero weights, which leaves every result as it
// is: rows and heads to multiples of 16, latents to 64, recurrence value heads to multiples of 32.
#include <math.h>
#include <string.h>

#include <algorithm>

#include "engine.h"
#include "mixers.h"
#include "project.h"
#include "weight_placer.h"

namespace onellm {

constexpr int kFuMaxSeq = 32768;   // positions of a sequence unless the caller says otherwise: the design has no limit
constexpr int kFuGateRank = 16;    // rank of the decay's projection when there are no weights to tell it
constexpr int kFuLatentTokens = 64;  // passes of at most this many tokens attend in latent space

struct FuposunLayerConfig {
    bool gla = false;
    int H = 0, dk = 0, dv = 0;
    int q_rank = 0, kv_rank = 0, window = 0;  // latent attention
    double scale = 1.0;
    double tau = 1.0;  // gla
    int gate_rank = kFuGateRank;
    enum { NONE, DENSE, MOE } ff_kind = NONE;
    int ff = 0;                                    // dense
    int experts = 0, top = 0, eff = 0, shared = 0;  // experts and their hidden size, the shared expert's
    double limit = 0.0, shared_limit = 0.0;
};

struct FuposunConfig {
    int vocab = 0, width = 0;
    double eps = 1e-6, residual_mult = 1.0, softcap = 1.0;
    std::vector<FuposunLayerConfig> layers;
};

static int read_mixer(const Json& m, const std::string& where, FuposunLayerConfig* l)
{
    const char* w = where.c_str();
    RC(json_int(m, "heads", w, &l->H));
    RC(json_int(m, "dim", w, &l->dk));
    RC(json_int(m, "vdim", w, &l->dv));
    ONELLM_REQUIRE(l->H > 0 && l->dk > 0 && l->dv > 0, ONELLM_ERR_IO, "config: sizes of %s", w);
    if (l->gla) {
        RC(json_float(m, "tau", w, &l->tau));
        ONELLM_REQUIRE(l->tau > 0.0, ONELLM_ERR_IO, "config: %s.tau", w);
        ONELLM_REQUIRE(l->dk <= 512 && l->dv <= 2048, ONELLM_ERR_UNSUPPORTED, "config: %s: key sizes above 512 and value sizes above 2048 are not supported", w);
        return ONELLM_OK;
    }
    const Json* mask;
    RC(json_int(m, "q_rank", w, &l->q_rank));
    RC(json_int(m, "kv_rank", w, &l->kv_rank));
    RC(json_float(m, "scale", w, &l->scale));
    RC(json_object(m, "mask", w, &mask));
    RC(json_int(*mask, "size", (where + ".mask").c_str(), &l->window));
    ONELLM_REQUIRE(l->q_rank > 0 && l->kv_rank > 0 && l->window > 0 && l->scale > 0.0, ONELLM_ERR_IO, "config: sizes of %s", w);
    ONELLM_REQUIRE(l->dk <= 256 && l->dv <= 256 && l->kv_rank <= 1024, ONELLM_ERR_UNSUPPORTED,
                   "config: %s: head sizes above 256 and latents above 1024 are not supported", w);
    return ONELLM_OK;
}

static int read_feed_forward(const Json& m, const std::string& where, FuposunLayerConfig* l)
{
    const Json* kind = m.find("kind");
    const char* w = where.c_str();
    if (kind && kind->text == "dense") {
        l->ff_kind = FuposunLayerConfig::DENSE;
        RC(json_int(m, "ff", w, &l->ff));
        ONELLM_REQUIRE(l->ff > 0, ONELLM_ERR_IO, "config: %s.ff", w);
        return ONELLM_OK;
    }
    ONELLM_REQUIRE(kind && kind->text == "moe", ONELLM_ERR_IO, "config: %s: unknown kind \"%s\"", w, kind ? kind->text.c_str() : "");
    l->ff_kind = FuposunLayerConfig::MOE;
    const Json *router, *expert, *shared;
    RC(json_object(m, "router", w, &router));
    RC(json_int(*router, "experts", (where + ".router").c_str(), &l->experts));
    RC(json_int(*router, "top", (where + ".router").c_str(), &l->top));
    RC(json_object(m, "expert", w, &expert));
    RC(json_int(*expert, "ff", (where + ".expert").c_str(), &l->eff));
    RC(json_float(*expert, "limit", (where + ".expert").c_str(), &l->limit));
    RC(json_object(m, "shared", w, &shared));
    RC(json_int(*shared, "ff", (where + ".shared").c_str(), &l->shared));
    RC(json_float(*shared, "limit", (where + ".shared").c_str(), &l->shared_limit));
    ONELLM_REQUIRE(l->experts > 0 && l->top > 0 && l->top <= l->experts && l->eff > 0 && l->shared > 0 && l->limit >= 0.0 && l->shared_limit >= 0.0,
                   ONELLM_ERR_IO, "config: sizes of %s", w);
    ONELLM_REQUIRE(l->experts <= 1024 && l->top <= 64, ONELLM_ERR_UNSUPPORTED, "config: %s: at most 64 of 1024 experts", w);
    return ONELLM_OK;
}

static int read_config(const Json& j, FuposunConfig* c)
{
    RC(json_int(j, "vocab", "config", &c->vocab));
    RC(json_int(j, "width", "config", &c->width));
    RC(json_float(j, "residual_mult", "config", &c->residual_mult));
    RC(json_float(j, "logit_softcap", "config", &c->softcap));
    const Json* norm;
    RC(json_object(j, "norm", "config", &norm));
    RC(json_float(*norm, "eps", "norm", &c->eps));
    const Json* layers = j.find("layers");
    ONELLM_REQUIRE(layers && layers->kind == Json::ARRAY && !layers->items.empty(), ONELLM_ERR_IO, "config: no \"layers\"");
    ONELLM_REQUIRE(c->vocab > 0 && c->width > 0 && c->softcap > 0.0, ONELLM_ERR_IO, "config: non-positive size");
    for (size_t i = 0; i < layers->items.size(); i++) {
        const Json& e = layers->items[i];
        const std::string where = "layers[" + std::to_string(i) + "]";
        FuposunLayerConfig l;
        const Json *type = e.find("type"), *mixer, *mlp = e.find("mlp");
        l.gla = type && type->text == "gla";
        ONELLM_REQUIRE(l.gla || (type && type->text == "latent_attention"), ONELLM_ERR_IO, "config: %s: unknown type \"%s\"", where.c_str(),
                       type ? type->text.c_str() : "");
        RC(json_object(e, "mixer", where.c_str(), &mixer));
        RC(read_mixer(*mixer, where + ".mixer", &l));
        if (mlp && !mlp->is_null()) RC(read_feed_forward(*mlp, where + ".mlp", &l));
        c->layers.push_back(l);
    }
    return ONELLM_OK;
}

struct FuposunWeights {
    // padded sizes; columns of the input matrix of the mixer [width, n_in]; the first group starts at 0
    int dk, dv, q_rank, kv_rank, n_in, n_out;
    int col_c, col_g;         // latent attention: latent, gate (the query latent is first)
    int col_k, col_v, col_a;  // gla: key, value, decay (the query is first; col_g: output gate)
    int ff, eff, shared, experts;
    float *norm1, *norm2;
    void *w_in, *w_out;
    float *q_norm, *kv_norm;         // latent attention
    void *w_uq, *w_uk, *w_kv;        // queries; keys per head [dk, kv_rank]; keys and values [kv_rank, H dk | H dv]
    float *A, *zb, *rnorm;           // gla
    void *w_gate, *w_up, *w_down;    // dense
    void *w_router, *e_gate, *e_up, *e_down, *s_gate, *s_up, *s_down;
};

struct FuposunMemory {
    void* ring;    // latent attention
    int R;         // its rows
    float* state;  // gla
};

struct Fuposun : Engine {
    FuposunConfig c;
    int dtype = ONELLM_BF16;
    int width = 0, vocab_p = 0;  // padded row width and vocabulary
    std::vector<FuposunWeights> weights;
    std::vector<FuposunMemory> mem;
    void *embed = nullptr, *head = nullptr;
    float *embed_norm = nullptr, *final_norm = nullptr;
    int* expert_count = nullptr;  // scratch of the routing, zero between passes

    // Buffers of a pass; one set for decode steps in the arena, one in the scratch of a context pass.
    struct Buffers {
        float *x, *router, *logits;
        void *h, *in, *cq, *q, *ql, *ol, *fresh, *kv, *cat, *act, *xs, *ys, *hn, *ws, *rec_work;
        Route route;
    };
    Buffers step = {};

    size_t esize() const { return dtype == ONELLM_F32 ? 4 : 2; }
    const char* design() const override { return "Fuposun"; }
    void carve(Carver& cv) override;
    int decode_layers(int step_bound, bool with_head) override;
    int context_layers(const ContextBatch& cb) override;
    int init_random(uint64_t seed, float std) override;

    bool in_latent_space(int tokens) const { return dtype == ONELLM_F32 || plain_kernels || tokens <= kFuLatentTokens; }
    // rows of the buffer of latents of a context pass that forms keys and values
    size_t joined_rows(const ContextBatch& cb, int window) const
    {
        size_t rows = cb.T;
        for (int b = 0; b < cb.B; b++) rows += std::min(cb.host_hist[b], window - 1);
        return rows;
    }
    void carve_buffers(Carver& cv, Buffers& b, size_t T, size_t n_rows, const ContextBatch* cb);

    // One pass: the tokens, where they are, and what the kernels size themselves by.
    struct Pass {
        Buffers& b;
        int T;
        TokenPositions tp;
        int max_new, max_hist, span;  // span: bound of the keys a query sees, before the window
        const ContextBatch* cb;
        const int* add_rows = nullptr;  // the experts' outputs of the layer before, not yet in the stream
        int add_n = 0;
    };
    int norm(Pass& p, const int* rows, int n_rows, const float* w, void* out);
    int latent_attention(size_t i, Pass& p);
    int gla(size_t i, Pass& p);
    int dense(size_t i, Pass& p);
    int experts(size_t i, Pass& p);
    int layers(Pass& p);
    int lm_head(Pass& p, const int* rows, int n_rows, float* out);
    int load(WeightPlacer& f);
    Projection projection(int M, const void* x, const void* W, void* y, int N, int K) const;
    // y = stream + residual_mult * x.W
    int add_to_stream(Pass& p, const void* x, const void* W, int K);
};

void Fuposun::carve_buffers(Carver& cv, Buffers& b, size_t T, size_t n_rows, const ContextBatch* cb)
{
    const size_t es = esize(), W = width;
    const bool latent = !cb || in_latent_space((int)T);
    size_t in = 0, cq = 0, q = 0, ql = 0, kv = 0, fresh = 0, cat = 0, act = 0, ws = 0, rec = 0, router = 0, slots = 0;
    int max_e = 0, max_tiles = 0;
    for (size_t i = 0; i < c.layers.size(); i++) {
        const FuposunLayerConfig& l = c.layers[i];
        const FuposunWeights& w = weights[i];
        in = std::max(in, T * w.n_in);
        cat = std::max(cat, T * w.n_out);
        if (l.gla) {
            if (cb) rec = std::max(rec, gated_recurrence_workspace(ONELLM_GR_KEYED, (int)T, l.H, w.dk, w.dv));
        } else {
            cq = std::max(cq, T * w.q_rank);
            q = std::max(q, T * l.H * w.dk);
            if (latent) {
                ql = std::max(ql, T * l.H * w.kv_rank);
                ws = std::max(ws, latent_attn_workspace((int)T, l.H, l.kv_rank));
                if (cb) fresh = std::max(fresh, T * w.kv_rank);
            } else {
                const size_t rows = joined_rows(*cb, l.window);
                fresh = std::max(fresh, rows * w.kv_rank);
                kv = std::max(kv, rows * l.H * (w.dk + w.dv));
            }
        }
        if (l.ff_kind == FuposunLayerConfig::DENSE) act = std::max(act, T * w.ff);
        if (l.ff_kind == FuposunLayerConfig::MOE) {
            act = std::max({act, T * w.shared, T * l.top * w.eff});
            router = std::max(router, T * w.experts);
            slots = std::max(slots, T * l.top);
            max_e = std::max(max_e, l.experts);
            max_tiles = std::max(max_tiles, route_max_tiles((int)T, l.experts, l.top));
        }
    }
    b.x = cv.take<float>(T * W);
    b.h = cv.take_bytes(T * W * es);
    b.in = cv.take_bytes(in * es);
    b.cq = cv.take_bytes(cq * es);
    b.q = cv.take_bytes(q * es);
    b.ql = cv.take_bytes(ql * es);
    b.ol = cv.take_bytes(ql * es);
    b.fresh = cv.take_bytes(fresh * es);
    b.kv = cv.take_bytes(kv * es);
    b.cat = cv.take_bytes(cat * es);
    b.act = cv.take_bytes(act * es);
    b.ws = cv.take_bytes(ws);
    b.rec_work = cv.take_bytes(rec);
    b.router = cv.take<float>(router);
    b.xs = T > 64 && dtype == ONELLM_BF16 ? cv.take_bytes(slots * W * es) : nullptr;
    b.ys = cv.take_bytes(slots * W * es);
    Route& r = b.route;
    r.slot = cv.take<int>(slots);
    r.slot_token = cv.take<int>(slots);
    r.slot_weight = cv.take<float>(slots);
    r.choice = cv.take<int>(slots);
    r.choice_weight = cv.take<float>(slots);
    r.off = cv.take<int>(max_e + 1);
    r.used = cv.take<int>(max_e);
    r.n_used = cv.take<int>(1);
    r.n_tiles = cv.take<int>(1);
    r.tile_group = cv.take<int>(max_tiles);
    r.tile_row = cv.take<int>(max_tiles);
    r.count = expert_count;
    b.hn = cv.take_bytes(n_rows * W * es);
    b.logits = cv.take<float>(n_rows * vocab_p);
}

void Fuposun::carve(Carver& cv)
{
    const size_t B = max_batch, W = width, es = esize();
    weights.assign(c.layers.size(), FuposunWeights{});
    mem.assign(c.layers.size(), FuposunMemory{});
    for (size_t i = 0; i < c.layers.size(); i++) {
        const FuposunLayerConfig& l = c.layers[i];
        FuposunWeights& w = weights[i];
        w.norm1 = cv.take<float>(W);
        w.dk = pad_to(l.dk, 16);
        if (l.gla) {
            w.dv = gated_recurrence_pad_dv(l.dv);
            w.col_k = l.H * w.dk;
            w.col_v = 2 * w.col_k;
            w.col_g = w.col_v + l.H * w.dv;
            w.col_a = w.col_g + l.H * w.dv;
            w.n_in = w.col_a + pad_to(l.gate_rank, 16);
            w.A = cv.take<float>((size_t)l.H * w.dk * l.gate_rank);
            w.zb = cv.take<float>((size_t)l.H * w.dk);
            w.rnorm = cv.take<float>(w.dv);
            mem[i].state = cv.take<float>(B * l.H * w.dk * w.dv);
        } else {
            w.dv = pad_to(l.dv, 16);
            w.q_rank = pad_to(l.q_rank, 16);
            w.kv_rank = latent_pad(l.kv_rank);
            w.col_c = w.q_rank;
            w.col_g = w.col_c + w.kv_rank;
            w.n_in = w.col_g + pad_to(l.H, 16);
            w.q_norm = cv.take<float>(w.q_rank);
            w.kv_norm = cv.take<float>(w.kv_rank);
            w.w_uq = cv.take_bytes((size_t)w.q_rank * l.H * w.dk * es);
            w.w_uk = cv.take_bytes((size_t)l.H * w.dk * w.kv_rank * es);
            w.w_kv = cv.take_bytes((size_t)w.kv_rank * l.H * (w.dk + w.dv) * es);
            mem[i].R = std::min(l.window, max_seq_len);
            mem[i].ring = cv.take_bytes(B * mem[i].R * w.kv_rank * es);
        }
        w.n_out = l.H * w.dv;
        w.w_in = cv.take_bytes(W * w.n_in * es);
        w.w_out = cv.take_bytes(W * w.n_out * es);
        if (l.ff_kind == FuposunLayerConfig::NONE) continue;
        w.norm2 = cv.take<float>(W);
        if (l.ff_kind == FuposunLayerConfig::DENSE) {
            w.ff = pad_to(l.ff, 16);
            w.w_gate = cv.take_bytes(W * w.ff * es);
            w.w_up = cv.take_bytes(W * w.ff * es);
            w.w_down = cv.take_bytes(W * w.ff * es);
        } else {
            w.eff = pad_to(l.eff, 16);
            w.shared = pad_to(l.shared, 16);
            w.experts = pad_to(l.experts, 8);
            w.w_router = cv.take_bytes(W * w.experts * es);
            const size_t e = W * w.eff * l.experts * es, s = W * w.shared * es;
            w.e_gate = cv.take_bytes(e);
            w.e_up = cv.take_bytes(e);
            w.e_down = cv.take_bytes(e);
            w.s_gate = cv.take_bytes(s);
            w.s_up = cv.take_bytes(s);
            w.s_down = cv.take_bytes(s);
        }
    }
    embed = cv.take_bytes((size_t)c.vocab * W * es);
    embed_norm = cv.take<float>(W);
    final_norm = cv.take<float>(W);
    head = cv.take_bytes(W * vocab_p * es);
    expert_count = cv.take<int>(1024);
    carve_buffers(cv, step, B, B, nullptr);
}

// ---- one layer ---------------------------------------------------------------------------------------------
Projection Fuposun::projection(int M, const void* x, const void* W, void* y, int N, int K) const
{
    Projection p;
    p.dtype = dtype;
    p.M = M;
    p.x = x;
    p.W = W;
    p.y = y;
    p.N = N;
    p.K = K;
    return p;
}

int Fuposun::add_to_stream(Pass& p, const void* x, const void* W, int K)
{
    Projection pj = projection(p.T, x, W, p.b.x, width, K);
    pj.f32 = 1;
    pj.resid = p.b.x;
    pj.scale = (float)c.residual_mult;
    return project(pj, stream);
}

// Norm of the stream, or of some rows of it; adds what the experts of the layer before left on its way.
int Fuposun::norm(Pass& p, const int* rows, int n_rows, const float* w, void* out)
{
    NormRows n = {dtype, p.b.x, rows, n_rows, w, nullptr, out, nullptr, (float)c.eps, 0.f, c.width, width, nullptr, nullptr, 0, 0.f};
    if (p.add_rows) {
        NormRows sum = n;
        sum.add = p.b.ys;
        sum.add_rows = p.add_rows;
        sum.add_n = p.add_n;
        sum.add_scale = (float)c.residual_mult;
        p.add_rows = nullptr;
        if (!rows) return norm_rows(sum, stream);
        sum.rows = nullptr;
        sum.n_rows = p.T;
        sum.out1 = nullptr;
        RC(norm_rows(sum, stream));
    }
    return norm_rows(n, stream);
}

int Fuposun::latent_attention(size_t i, Pass& p)
{
    const FuposunLayerConfig& l = c.layers[i];
    const FuposunWeights& w = weights[i];
    Buffers& b = p.b;
    const size_t es = esize();
    auto at = [es](void* base, int col) { return static_cast<void*>(static_cast<char*>(base) + (size_t)col * es); };
    const bool latent = !p.cb || in_latent_space(p.T);
    const int hk = l.H * w.dk, hc = l.H * w.kv_rank, kv_ld = l.H * (w.dk + w.dv);
    RC(project(projection(p.T, b.h, w.w_in, b.in, w.n_in, width), stream));
    LatentAttn a = {};
    a.dtype = dtype;
    a.H = l.H;
    a.rank = l.kv_rank;
    a.window = l.window;
    a.R = mem[i].R;
    a.ring = mem[i].ring;
    a.fresh = b.fresh;
    a.joined = !latent;
    a.q_src = b.in;
    a.kv_src = at(b.in, w.col_c);
    a.ld = w.n_in;
    a.q_w = w.q_norm;
    a.kv_w = w.kv_norm;
    a.q_width = l.q_rank;
    a.q_ld = w.q_rank;
    a.q_out = b.cq;
    a.eps = (float)c.eps;
    RC(latent_store(a, p.tp, p.T, p.max_hist, stream));
    RC(project(projection(p.T, b.cq, w.w_uq, b.q, hk, w.q_rank), stream));
    if (latent) {
        RowGroups heads = {};
        heads.n = l.H;
        heads.w_stride = (long)w.dk * w.kv_rank;
        heads.x_stride = w.dk;
        heads.y_stride = w.kv_rank;
        Projection in = projection(p.T, b.q, w.w_uk, b.ql, w.kv_rank, w.dk);
        in.ldx = hk;
        in.ldy = hc;
        in.ldw = w.kv_rank;
        in.groups = &heads;
        RC(project(in, stream));
        a.q = b.ql;
        a.scale = (float)l.scale;
        a.gate = at(b.in, w.col_g);
        a.gate_ld = w.n_in;
        a.out = b.ol;
        a.out_scale = 1.f;
        RC(latent_attn(a, p.tp, p.T, p.span, plain_kernels, b.ws, stream));
        heads.w_stride = w.dv;
        heads.x_stride = w.kv_rank;
        heads.y_stride = w.dv;
        Projection out = projection(p.T, b.ol, at(w.w_kv, hk), b.cat, w.dv, w.kv_rank);
        out.ldx = hc;
        out.ldy = w.n_out;
        out.ldw = kv_ld;
        out.groups = &heads;
        RC(project(out, stream));
    } else {
        const size_t rows = joined_rows(*p.cb, l.window);
        RC(project(projection((int)rows, b.fresh, w.w_kv, b.kv, kv_ld, w.kv_rank), stream));
        RC(window_attn({l.H, w.dk, w.dv, l.window, b.q, hk, b.kv, kv_ld, (long)rows, (float)l.scale, at(b.in, w.col_g), w.n_in, b.cat, w.n_out, 1.f}, p.tp,
                       p.max_new, stream));
    }
    if (p.cb) RC(latent_keep(a, p.tp, p.max_new, stream));
    return add_to_stream(p, b.cat, w.w_out, w.n_out);
}

int Fuposun::gla(size_t i, Pass& p)
{
    const FuposunLayerConfig& l = c.layers[i];
    const FuposunWeights& w = weights[i];
    Buffers& b = p.b;
    const size_t es = esize();
    auto at = [es](void* base, int col) { return static_cast<void*>(static_cast<char*>(base) + (size_t)col * es); };
    RC(project(projection(p.T, b.h, w.w_in, b.in, w.n_in, width), stream));
    GatedRecurrence g = {};
    g.dtype = dtype;
    g.kind = ONELLM_GR_KEYED;
    g.H = l.H;
    g.dk = w.dk;
    g.dv = w.dv;
    g.q = b.in;
    g.k = at(b.in, w.col_k);
    g.v = at(b.in, w.col_v);
    g.g = at(b.in, w.col_g);
    g.r = at(b.in, w.col_a);
    g.rank = l.gate_rank;
    g.A = w.A;
    g.zb = w.zb;
    g.inv_tau = (float)(1.0 / l.tau);
    g.q_scale = (float)(1.0 / sqrt((double)l.dk));
    g.ld = w.n_in;
    g.w = w.rnorm;
    g.eps = (float)c.eps;
    g.norm_width = l.dv;
    g.state = mem[i].state;
    g.out = b.cat;
    g.out_ld = w.n_out;
    g.out_scale = 1.f;
    g.work = b.rec_work;
    RC(gated_recurrence(g, p.tp, p.tp.B, p.T, stream));
    return add_to_stream(p, b.cat, w.w_out, w.n_out);
}

int Fuposun::dense(size_t i, Pass& p)
{
    const FuposunWeights& w = weights[i];
    Projection gu = projection(p.T, p.b.h, w.w_gate, p.b.act, w.ff, width);
    gu.W2 = w.w_up;
    gu.act = GATE_SILU;
    RC(project(gu, stream));
    return add_to_stream(p, p.b.act, w.w_down, w.ff);
}

int Fuposun::experts(size_t i, Pass& p)
{
    const FuposunLayerConfig& l = c.layers[i];
    const FuposunWeights& w = weights[i];
    Buffers& b = p.b;
    Projection z = projection(p.T, b.h, w.w_router, b.router, w.experts, width);
    z.f32 = 1;
    RC(project(z, stream));
    Route r = b.route;
    r.T = p.T;
    r.experts = l.experts;
    r.top = l.top;
    r.logits = b.router;
    r.ld = w.experts;
    r.dtype = dtype;
    r.x = b.h;
    r.xs = b.xs;
    r.ld_x = width;
    RC(route(r, stream));
    const bool tiled = b.xs != nullptr;  // rows copied into expert order; else the projection picks them
    RowGroups g = {};
    g.n = tiled ? l.experts : std::min(l.experts, p.T * l.top);
    g.used = tiled ? nullptr : r.used;
    g.n_used = tiled ? nullptr : r.n_used;
    g.off = r.off;
    g.x_rows = tiled ? nullptr : r.slot_token;
    g.row_scale = r.slot_weight;  // the weight of an expert goes into its gate and up products
    g.w_stride = (long)width * w.eff;
    g.tile_group = r.tile_group;
    g.tile_row = r.tile_row;
    g.n_tiles = r.n_tiles;
    g.max_tiles = route_max_tiles(p.T, l.experts, l.top);
    g.weights = l.experts;
    g.rows = (long)p.T * l.top;
    Projection gu = projection(p.T, tiled ? b.xs : b.h, w.e_gate, b.act, w.eff, width);
    gu.W2 = w.e_up;
    gu.act = GATE_CLAMPED;
    gu.limit = (float)l.limit;
    gu.groups = &g;
    RC(project(gu, stream));
    Projection down = projection(p.T, b.act, w.e_down, b.ys, width, w.eff);
    g.x_rows = nullptr;
    g.row_scale = nullptr;
    down.groups = &g;
    RC(project(down, stream));
    // the shared expert, straight into the stream
    Projection sgu = projection(p.T, b.h, w.s_gate, b.act, w.shared, width);
    sgu.W2 = w.s_up;
    sgu.act = GATE_CLAMPED;
    sgu.limit = (float)l.shared_limit;
    RC(project(sgu, stream));
    RC(add_to_stream(p, b.act, w.s_down, w.shared));
    p.add_rows = r.slot;
    p.add_n = l.top;
    return ONELLM_OK;
}

int Fuposun::layers(Pass& p)
{
    for (size_t i = 0; i < c.layers.size(); i++) {
        const FuposunLayerConfig& l = c.layers[i];
        const FuposunWeights& w = weights[i];
        RC(norm(p, nullptr, p.T, w.norm1, p.b.h));
        RC(l.gla ? gla(i, p) : latent_attention(i, p));
        if (l.ff_kind == FuposunLayerConfig::NONE) continue;
        RC(norm(p, nullptr, p.T, w.norm2, p.b.h));
        RC(l.ff_kind == FuposunLayerConfig::DENSE ? dense(i, p) : experts(i, p));
    }
    return ONELLM_OK;
}

// Final norm, head and soft cap of some rows of the stream (rows NULL: all); logits in float, [n_rows, vocab].
int Fuposun::lm_head(Pass& p, const int* rows, int n_rows, float* out)
{
    RC(norm(p, rows, n_rows, final_norm, p.b.hn));
    Projection pj = projection(n_rows, p.b.hn, head, p.b.logits, vocab_p, width);
    pj.f32 = 1;
    RC(project(pj, stream));
    return softcap(p.b.logits, vocab_p, out, n_rows, c.vocab, (float)c.softcap, stream);
}

int Fuposun::decode_layers(int step_bound, bool with_head)
{
    RC(embedding_norm_launch(dtype, d_ids, step.x, embed, embed_norm, (float)c.eps, batch, c.width, width, c.vocab, d_bad_id, stream));
    Pass p = {step, batch, {nullptr, nullptr, batch, d_step, d_step_off}, 1, 0, step_bound, nullptr};
    RC(layers(p));
    return with_head ? lm_head(p, nullptr, batch, static_cast<float*>(logits)) : ONELLM_OK;
}

int Fuposun::context_layers(const ContextBatch& cb)
{
    Buffers b = {};
    Carver sizing{nullptr};
    carve_buffers(sizing, b, cb.T, cb.n_rows, &cb);
    RC(ensure_scratch(align_up(sizing.off, 256)));
    Carver real{scratch};
    carve_buffers(real, b, cb.T, cb.n_rows, &cb);
    const int max_hist = *std::max_element(cb.host_hist, cb.host_hist + cb.B);
    RC(embedding_norm_launch(dtype, d_prompt, b.x, embed, embed_norm, (float)c.eps, (int)cb.T, c.width, width, c.vocab, d_bad_id, stream));
    Pass p = {b, (int)cb.T, {cb.cu, cb.hist, cb.B, nullptr, nullptr}, cb.P, max_hist, max_hist + cb.P, &cb};
    RC(layers(p));
    RC(lm_head(p, cb.rows, cb.n_rows, static_cast<float*>(cb.logits)));
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}

// ---- weights -----------------------------------------------------------------------------------------------
int Fuposun::load(WeightPlacer& f)
{
    const int D = c.width;
    const size_t es = esize();
    auto behind = [es](void* base, size_t elements) { return static_cast<void*>(static_cast<char*>(base) + elements * es); };
    RC(f.place("embed", embed, width, 0, 0, c.vocab, c.vocab, c.vocab, D, D, D, false));
    RC(f.vec("embed.norm", embed_norm, D));
    RC(f.vec("final.norm", final_norm, D));
    RC(f.columns("head", head, vocab_p, 0, c.vocab, D));
    for (size_t i = 0; i < c.layers.size(); i++) {
        const FuposunLayerConfig& l = c.layers[i];
        const FuposunWeights& w = weights[i];
        const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.";
        const int hk = l.H * l.dk, hv = l.H * l.dv;
        RC(f.vec(p + "norm1", w.norm1, D));
        if (l.gla) {
            RC(f.place(m + "q", w.w_in, w.n_in, 0, 0, hk, l.dk, w.dk, D, D, D));
            RC(f.place(m + "k", w.w_in, w.n_in, 0, w.col_k, hk, l.dk, w.dk, D, D, D));
            RC(f.place(m + "v", w.w_in, w.n_in, 0, w.col_v, hv, l.dv, w.dv, D, D, D));
            RC(f.place(m + "g", w.w_in, w.n_in, 0, w.col_g, hv, l.dv, w.dv, D, D, D));
            RC(f.columns(m + "a1", w.w_in, w.n_in, w.col_a, l.gate_rank, D));
            RC(f.rows_f32(m + "a2", w.A, l.gate_rank, hk, l.dk, w.dk, l.gate_rank));
            RC(f.vec(m + "a2.b", w.zb, hk, l.dk, w.dk));
            RC(f.vec(m + "norm", w.rnorm, l.dv));
        } else {
            const int kv_ld = l.H * (w.dk + w.dv);
            RC(f.columns(m + "dq", w.w_in, w.n_in, 0, l.q_rank, D));
            RC(f.columns(m + "dkv", w.w_in, w.n_in, w.col_c, l.kv_rank, D));
            RC(f.columns(m + "g", w.w_in, w.n_in, w.col_g, l.H, D));
            RC(f.vec(m + "dq.norm", w.q_norm, l.q_rank));
            RC(f.vec(m + "dkv.norm", w.kv_norm, l.kv_rank));
            RC(f.place(m + "uq", w.w_uq, l.H * w.dk, 0, 0, hk, l.dk, w.dk, l.q_rank, l.q_rank, l.q_rank));
            RC(f.place(m + "uk", w.w_uk, w.kv_rank, 0, 0, hk, l.dk, w.dk, l.kv_rank, l.kv_rank, l.kv_rank, false));
            RC(f.place(m + "uk", w.w_kv, kv_ld, 0, 0, hk, l.dk, w.dk, l.kv_rank, l.kv_rank, l.kv_rank));
            RC(f.place(m + "uv", w.w_kv, kv_ld, 0, l.H * w.dk, hv, l.dv, w.dv, l.kv_rank, l.kv_rank, l.kv_rank));
        }
        RC(f.place(m + "o", w.w_out, width, 0, 0, D, D, D, hv, l.dv, w.dv));
        if (l.ff_kind == FuposunLayerConfig::NONE) continue;
        const std::string n = p + "mlp.";
        RC(f.vec(p + "norm2", w.norm2, D));
        if (l.ff_kind == FuposunLayerConfig::DENSE) {
            RC(f.columns(n + "gate", w.w_gate, w.ff, 0, l.ff, D));
            RC(f.columns(n + "up", w.w_up, w.ff, 0, l.ff, D));
            RC(f.columns(n + "down", w.w_down, width, 0, D, l.ff));
            continue;
        }
        RC(f.columns(n + "router", w.w_router, w.experts, 0, l.experts, D));
        for (int e = 0; e < l.experts; e++) {
            const std::string x = n + "e" + std::to_string(e) + ".";
            const size_t first = (size_t)e * width * w.eff;
            RC(f.columns(x + "gate", behind(w.e_gate, first), w.eff, 0, l.eff, D));
            RC(f.columns(x + "up", behind(w.e_up, first), w.eff, 0, l.eff, D));
            RC(f.columns(x + "down", behind(w.e_down, first), width, 0, D, l.eff));
        }
        RC(f.columns(n + "shared.gate", w.s_gate, w.shared, 0, l.shared, D));
        RC(f.columns(n + "shared.up", w.s_up, w.shared, 0, l.shared, D));
        RC(f.columns(n + "shared.down", w.s_down, width, 0, D, l.shared));
    }
    weights_ready = true;
    return ONELLM_OK;
}

// Random weights of the configured shape (padding included: sizes are then what the kernels see), states that forget slowly.
int Fuposun::init_random(uint64_t seed, float std)
{
    uint64_t tag = 1;
    auto normal = [&](void* w, size_t rows, size_t cols) { return init_normal(dtype, w, rows, cols, cols, 0, 0, seed, tag++, 0.f, std, stream); };
    auto fill = [&](float* w, size_t n, float v) { return init_normal(ONELLM_F32, w, 1, n, n, 0, 0, seed, 0, v, 0.f, stream); };
    for (size_t i = 0; i < c.layers.size(); i++) {
        const FuposunLayerConfig& l = c.layers[i];
        const FuposunWeights& w = weights[i];
        RC(fill(w.norm1, width, 1.f));
        RC(normal(w.w_in, width, w.n_in));
        RC(normal(w.w_out, w.n_out, width));
        if (l.gla) {
            RC(init_normal(ONELLM_F32, w.A, (size_t)l.H * w.dk, l.gate_rank, l.gate_rank, 0, 0, seed, tag++, 0.f, std, stream));
            RC(fill(w.zb, (size_t)l.H * w.dk, 2.f));
            RC(fill(w.rnorm, w.dv, 1.f));
        } else {
            RC(fill(w.q_norm, w.q_rank, 1.f));
            RC(fill(w.kv_norm, w.kv_rank, 1.f));
            RC(normal(w.w_uq, w.q_rank, (size_t)l.H * w.dk));
            RC(normal(w.w_uk, (size_t)l.H * w.dk, w.kv_rank));
            RC(normal(w.w_kv, w.kv_rank, (size_t)l.H * (w.dk + w.dv)));
        }
        if (l.ff_kind == FuposunLayerConfig::NONE) continue;
        RC(fill(w.norm2, width, 1.f));
        if (l.ff_kind == FuposunLayerConfig::DENSE) {
            RC(normal(w.w_gate, width, w.ff));
            RC(normal(w.w_up, width, w.ff));
            RC(normal(w.w_down, w.ff, width));
        } else {
            RC(normal(w.w_router, width, w.experts));
            RC(normal(w.e_gate, (size_t)l.experts * width, w.eff));
            RC(normal(w.e_up, (size_t)l.experts * width, w.eff));
            RC(normal(w.e_down, (size_t)l.experts * w.eff, width));
            RC(normal(w.s_gate, width, w.shared));
            RC(normal(w.s_up, width, w.shared));
            RC(normal(w.s_down, w.shared, width));
        }
    }
    RC(normal(embed, c.vocab, width));
    RC(normal(head, width, vocab_p));
    RC(fill(embed_norm, width, 1.f));
    RC(fill(final_norm, width, 1.f));
    ONELLM_CUDA(cudaStreamSynchronize(stream));
    weights_ready = true;
    return ONELLM_OK;
}

// What the configuration leaves to the shapes of the tensors.
static int read_shapes(const SafeTensors& file, FuposunConfig* c)
{
    for (size_t i = 0; i < c->layers.size(); i++) {
        FuposunLayerConfig& l = c->layers[i];
        if (!l.gla) continue;
        const std::string name = "l" + std::to_string(i) + ".mix.a1";
        const SafeTensor* t = file.find(name);
        ONELLM_REQUIRE(t, ONELLM_ERR_IO, "no tensor %s", name.c_str());
        ONELLM_REQUIRE(t->shape.size() == 2 && t->shape[0] > 0 && t->shape[0] <= 1024, ONELLM_ERR_IO, "tensor %s: a matrix of 1 to 1024 rows", name.c_str());
        l.gate_rank = (int)t->shape[0];
    }
    return ONELLM_OK;
}

static int open_fuposun(Fuposun* m, const Json& config, const std::string& folder, const ModelOptions& opt)
{
    RC(read_config(config, &m->c));
    ONELLM_REQUIRE(opt.max_batch >= 1 && opt.max_batch <= 64, ONELLM_ERR_ARG, "model_open: max_batch %d outside [1, 64]", opt.max_batch);
    WeightPlacer placer(opt.dtype, nullptr);
    if (!folder.empty()) {
        RC(placer.file.open(folder + "/model.safetensors"));
        RC(read_shapes(placer.file, &m->c));
    }
    m->dtype = opt.dtype;
    m->vocab = m->c.vocab;
    m->width = pad_to(m->c.width, 16);
    m->vocab_p = pad_to(m->c.vocab, 8);
    m->logits_dtype = ONELLM_F32;
    m->eos_id = -1;  // the design names no end-of-sequence token
    m->max_batch = opt.max_batch;
    m->max_seq_len = opt.max_seq_len > 0 ? opt.max_seq_len : kFuMaxSeq;
    m->span_cap = 1;
    for (const FuposunLayerConfig& l : m->c.layers) m->span_cap = std::max(m->span_cap, l.window);
    RC(m->allocate());  // the arena starts as zeros: so do the padding of the weights, the rings and the states
    if (folder.empty()) return ONELLM_OK;
    placer.stream = m->stream;
    return m->load(placer);
}

static int make_fuposun(const Json& config, const std::string& folder, const ModelOptions& opt, Engine** out)
{
    Fuposun* m = new Fuposun();
    const int rc = open_fuposun(m, config, folder, opt);
    if (rc) {
        delete m;
        return rc;
    }
    *out = m;
    return ONELLM_OK;
}

static const ModelRegistration register_fuposun("Fuposun", make_fuposun);

}  // namespace onellm
