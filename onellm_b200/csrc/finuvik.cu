// The Finuvik design: a decoder whose layers put two sequence mixers and a feed-forward side by side on one residual
// stream,
//     x <- x + left_scale * attention(n1(x)) + right_scale * recurrence(n1(x)) + ff(n2(x)),
// with learned positions, zero-centred RMS norms, grouped-query attention that has a logarithmic query temperature and a
// logarithmic distance penalty instead of a rotation, an HGRN2 recurrence and a ReLU-gated feed-forward (a layer may
// have none).  Layers may share the weights of another layer; every layer run has its own cache and state.
//
// The parallel form sets the launches of a layer.  All branch inputs come from one pass over the stream (norm_rows), all
// mixer projections are one matrix [width, q | k | v | q' | f | v'], and all branch outputs are columns of one buffer
//     cat = [ left_scale * attention | right_scale * recurrence | relu(gate) * up ]
// whose product with the stacked output weights [W_o ; W_o' ; W_down] is added to the float residual stream in the
// epilogue of one projection: six launches per layer (norm, mixer projection, gate/up, attention, recurrence, output),
// seven when the decode attention is split.
//
// Sizes that the kernels do not take as they are get padded in memory with zero weights, which leaves every result as
// it is: rows to multiples of 16, attention heads to multiples of 16, recurrence value heads to multiples of 32.
#include <math.h>
#include <string.h>

#include <algorithm>

#include "engine.h"
#include "mixers.h"
#include "model_files.h"
#include "project.h"
#include "weight_placer.h"

namespace onellm {

struct FinuvikLayerConfig {
    int weights_of = -1;  // the layer whose tensors are used (itself, or the one named)
    int H = 0, G = 0, dk = 0, dv = 0;
    double scale = 1.0, temp_coef = 0.0, temp_every = 1.0;
    int RH = 0, rk = 0, rv = 0;
    double left_scale = 1.0, right_scale = 1.0;
    int ff = 0;  // 0: no feed-forward
};

struct FinuvikConfig {
    int vocab = 0, width = 0, max_positions = 0;
    double eps = 1e-6;
    std::vector<FinuvikLayerConfig> layers;
};

static int read_mixer(const Json& m, const std::string& where, FinuvikLayerConfig* l)
{
    const Json *left, *right;
    const std::string lw = where + ".left", rw = where + ".right";
    RC(json_object(m, "left", where.c_str(), &left));
    RC(json_object(m, "right", where.c_str(), &right));
    RC(json_int(*left, "heads", lw.c_str(), &l->H));
    RC(json_int(*left, "kv_heads", lw.c_str(), &l->G));
    RC(json_int(*left, "dim", lw.c_str(), &l->dk));
    RC(json_int(*left, "vdim", lw.c_str(), &l->dv));
    RC(json_float(*left, "scale", lw.c_str(), &l->scale));
    const Json* temp = left->find("q_temp");
    if (temp && !temp->is_null()) {
        RC(json_float(*temp, "coef", (lw + ".q_temp").c_str(), &l->temp_coef));
        RC(json_float(*temp, "every", (lw + ".q_temp").c_str(), &l->temp_every));
    }
    RC(json_int(*right, "heads", rw.c_str(), &l->RH));
    RC(json_int(*right, "dim", rw.c_str(), &l->rk));
    RC(json_int(*right, "vdim", rw.c_str(), &l->rv));
    RC(json_float(m, "left_scale", where.c_str(), &l->left_scale));
    RC(json_float(m, "right_scale", where.c_str(), &l->right_scale));
    ONELLM_REQUIRE(l->H > 0 && l->G > 0 && l->H % l->G == 0 && l->dk > 0 && l->dv > 0 && l->RH > 0 && l->rk > 0 && l->rv > 0 &&
                       l->temp_every > 0.0,
                   ONELLM_ERR_IO, "config: sizes of %s", where.c_str());
    ONELLM_REQUIRE(l->dk <= 256 && l->dv <= 256 && l->rk <= 256 && l->rv <= 256, ONELLM_ERR_UNSUPPORTED,
                   "config: %s: head sizes above 256 are not supported", where.c_str());
    return ONELLM_OK;
}

static int read_config(const Json& j, FinuvikConfig* c)
{
    RC(json_int(j, "vocab", "config", &c->vocab));
    RC(json_int(j, "width", "config", &c->width));
    RC(json_int(j, "max_positions", "config", &c->max_positions));
    const Json* norm;
    RC(json_object(j, "norm", "config", &norm));
    RC(json_float(*norm, "eps", "norm", &c->eps));
    const Json* layers = j.find("layers");
    ONELLM_REQUIRE(layers && layers->kind == Json::ARRAY && !layers->items.empty(), ONELLM_ERR_IO, "config: no \"layers\"");
    ONELLM_REQUIRE(c->vocab > 0 && c->width > 0 && c->max_positions > 0, ONELLM_ERR_IO, "config: non-positive size");
    for (size_t i = 0; i < layers->items.size(); i++) {
        const Json& e = layers->items[i];
        const std::string where = "layers[" + std::to_string(i) + "]";
        FinuvikLayerConfig l;
        const Json *type = e.find("type"), *mixer, *mlp = e.find("mlp"), *of = e.find("weights_of");
        ONELLM_REQUIRE(type && type->text == "parallel", ONELLM_ERR_IO, "config: %s: unknown type \"%s\"", where.c_str(), type ? type->text.c_str() : "");
        RC(json_object(e, "mixer", where.c_str(), &mixer));
        RC(read_mixer(*mixer, where + ".mixer", &l));
        if (mlp && !mlp->is_null()) {
            const Json* kind = mlp->find("kind");
            ONELLM_REQUIRE(kind && kind->text == "dense", ONELLM_ERR_IO, "config: %s.mlp: unknown kind \"%s\"", where.c_str(), kind ? kind->text.c_str() : "");
            RC(json_int(*mlp, "ff", (where + ".mlp").c_str(), &l.ff));
            ONELLM_REQUIRE(l.ff > 0, ONELLM_ERR_IO, "config: %s.mlp.ff", where.c_str());
        }
        l.weights_of = (int)i;
        if (of && !of->is_null()) {
            RC(json_int(e, "weights_of", where.c_str(), &l.weights_of));
            ONELLM_REQUIRE(l.weights_of >= 0 && l.weights_of < (int)layers->items.size(), ONELLM_ERR_IO, "config: %s.weights_of", where.c_str());
        }
        c->layers.push_back(l);
    }
    for (size_t i = 0; i < c->layers.size(); i++) {
        int j0 = c->layers[i].weights_of;
        for (size_t hop = 0; hop < c->layers.size() && c->layers[j0].weights_of != j0; hop++) j0 = c->layers[j0].weights_of;
        const FinuvikLayerConfig &a = c->layers[i], &b = c->layers[j0];
        ONELLM_REQUIRE(b.weights_of == j0, ONELLM_ERR_IO, "config: layers[%zu].weights_of leads in a circle", i);
        ONELLM_REQUIRE(a.H == b.H && a.G == b.G && a.dk == b.dk && a.dv == b.dv && a.RH == b.RH && a.rk == b.rk && a.rv == b.rv && a.ff == b.ff,
                       ONELLM_ERR_IO, "config: layers[%zu] uses the weights of layer %d but has other sizes", i, j0);
        c->layers[i].weights_of = j0;
    }
    return ONELLM_OK;
}

// The tensors of one layer (shared by the layers that name it).
struct FinuvikWeights {
    // padded sizes and the columns of the packed matrices
    int dk, dv, rk, rv, ff;
    int col_k, col_v, col_rq, col_rf, col_rv, n_mix;  // mixer projection [width, n_mix]; q starts at 0
    int cat_r, cat_f, n_cat;                          // output projection [n_cat, width]; attention starts at 0
    float *norm1, *norm2, *r1, *r2, *zb, *lower, *rnorm;
    float *q_factor, *penalty;
    void *w_mix, *w_gate, *w_up, *w_out;
};

struct FinuvikMemory {
    void *k, *v;
    float* state;
};

struct Finuvik : Engine {
    FinuvikConfig c;
    int dtype = ONELLM_BF16;
    int width = 0, vocab_p = 0;  // padded row width and vocabulary
    int max_mix = 0, max_cat = 0, max_ws_heads = 0, max_ws_dv = 0;
    std::vector<FinuvikWeights> weights;  // per layer; only the ones with tensors of their own are filled
    std::vector<FinuvikMemory> mem;       // per layer run
    void *embed = nullptr, *pos = nullptr, *head = nullptr;
    float* final_norm = nullptr;
    // decode activations
    float *x = nullptr, *logits_p = nullptr;
    void *h1 = nullptr, *h2 = nullptr, *mix = nullptr, *cat = nullptr, *ws = nullptr;

    size_t esize() const { return dtype == ONELLM_F32 ? 4 : 2; }
    const char* design() const override { return "Finuvik"; }
    void carve(Carver& cv) override;
    int decode_layers(int step_bound, bool with_head) override;
    int context_layers(const ContextBatch& cb) override;
    int init_random(uint64_t seed, float std) override;

    struct Buffers {
        float* x;
        void *h1, *h2, *mix, *cat;
        void* rec_work;  // context pass only
    };
    int layer(size_t i, const Buffers& buf, int tokens, const TokenPositions& tp, int max_new, int step_bound);
    int norm(float* stream_rows, const int* rows, int n_rows, const float* w1, const float* w2, void* out1, void* out2);
    int lm_head(float* stream_rows, const int* rows, int n_rows, void* hn, float* padded, float* out);
    int load(const std::string& folder);
    int finalize();
    bool own(size_t i) const { return c.layers[i].weights_of == (int)i; }
};

void Finuvik::carve(Carver& cv)
{
    const size_t B = max_batch, W = width, es = esize();
    weights.resize(c.layers.size());
    mem.resize(c.layers.size());
    for (size_t i = 0; i < c.layers.size(); i++) {
        const FinuvikLayerConfig& l = c.layers[i];
        FinuvikWeights& w = weights[i];
        w.dk = pad_to(l.dk, 16);
        w.dv = pad_to(l.dv, 16);
        w.rk = pad_to(l.rk, 16);
        w.rv = pad_to(l.rv, 32);
        w.ff = pad_to(l.ff, 16);
        w.col_k = l.H * w.dk;
        w.col_v = w.col_k + l.G * w.dk;
        w.col_rq = w.col_v + l.G * w.dv;
        w.col_rf = w.col_rq + l.RH * w.rk;
        w.col_rv = w.col_rf + l.RH * w.rk;
        w.n_mix = w.col_rv + l.RH * w.rv;
        w.cat_r = l.H * w.dv;
        w.cat_f = w.cat_r + l.RH * w.rv;
        w.n_cat = w.cat_f + w.ff;
        max_mix = std::max(max_mix, w.n_mix);
        max_cat = std::max(max_cat, w.n_cat);
        max_ws_heads = std::max(max_ws_heads, l.H);
        max_ws_dv = std::max(max_ws_dv, w.dv);
        if (own(i)) {
            w.norm1 = cv.take<float>(W);
            w.norm2 = cv.take<float>(W);
            w.r1 = cv.take<float>(l.H);
            w.r2 = cv.take<float>(l.H);
            w.zb = cv.take<float>((size_t)l.RH * w.rk);
            w.lower = cv.take<float>((size_t)l.RH * w.rk);
            w.rnorm = cv.take<float>(w.rv);
            w.q_factor = cv.take<float>(max_seq_len);
            w.penalty = cv.take<float>((size_t)l.H * max_seq_len);
            w.w_mix = cv.take_bytes(W * w.n_mix * es);
            w.w_gate = w.ff ? cv.take_bytes(W * w.ff * es) : nullptr;
            w.w_up = w.ff ? cv.take_bytes(W * w.ff * es) : nullptr;
            w.w_out = cv.take_bytes(W * w.n_cat * es);
        }
        mem[i].k = cv.take_bytes(B * l.G * max_seq_len * w.dk * es);
        mem[i].v = cv.take_bytes(B * l.G * max_seq_len * w.dv * es);
        mem[i].state = cv.take<float>(B * l.RH * w.rk * w.rv);
    }
    embed = cv.take_bytes((size_t)c.vocab * W * es);
    pos = cv.take_bytes((size_t)c.max_positions * W * es);
    final_norm = cv.take<float>(W);
    head = cv.take_bytes(W * vocab_p * es);
    x = cv.take<float>(B * W);
    h1 = cv.take_bytes(B * W * es);
    h2 = cv.take_bytes(B * W * es);
    mix = cv.take_bytes(B * max_mix * es);
    cat = cv.take_bytes(B * max_cat * es);
    logits_p = vocab_p == c.vocab ? nullptr : cv.take<float>(B * vocab_p);
    ws = cv.take_bytes(biased_attn_decode_workspace((int)B, max_ws_heads, max_ws_dv));
}

int Finuvik::norm(float* stream_rows, const int* rows, int n_rows, const float* w1, const float* w2, void* out1, void* out2)
{
    return norm_rows({dtype, stream_rows, rows, n_rows, w1, w2, out1, out2, (float)c.eps, 1.f, c.width, width, nullptr, nullptr, 0, 0.f}, stream);
}

// One layer over `tokens` tokens: a context pass (tp.cu) or a decode step.
int Finuvik::layer(size_t i, const Buffers& buf, int tokens, const TokenPositions& tp, int max_new, int step_bound)
{
    const FinuvikLayerConfig& l = c.layers[i];
    const FinuvikWeights& w = weights[l.weights_of];
    const size_t es = esize();
    auto at = [es](void* base, int col) { return static_cast<void*>(static_cast<char*>(base) + (size_t)col * es); };
    RC(norm(buf.x, nullptr, tokens, w.norm1, w.norm2, buf.h1, w.ff ? buf.h2 : nullptr));
    Projection pj;
    pj.dtype = dtype;
    pj.M = tokens;
    pj.x = buf.h1;
    pj.W = w.w_mix;
    pj.y = buf.mix;
    pj.N = w.n_mix;
    pj.K = width;
    RC(project(pj, stream));
    if (w.ff) {
        pj.x = buf.h2;
        pj.W = w.w_gate;
        pj.W2 = w.w_up;
        pj.y = at(buf.cat, w.cat_f);
        pj.ldy = w.n_cat;
        pj.N = w.ff;
        pj.act = GATE_RELU;
        RC(project(pj, stream));
    }
    BiasedAttn a = {};
    a.dtype = dtype;
    a.H = l.H;
    a.G = l.G;
    a.dk = w.dk;
    a.dv = w.dv;
    a.q = buf.mix;
    a.k = at(buf.mix, w.col_k);
    a.v = at(buf.mix, w.col_v);
    a.ld = w.n_mix;
    a.k_cache = mem[i].k;
    a.v_cache = mem[i].v;
    a.S = max_seq_len;
    a.q_factor = w.q_factor;
    a.penalty = w.penalty;
    a.out = buf.cat;
    a.out_ld = w.n_cat;
    a.out_scale = (float)l.left_scale;
    if (!tp.cu && dtype == ONELLM_BF16 && !plain_kernels) {
        RC(biased_attn_decode(a, tp, step_bound, ws, stream));
    } else {
        RC(biased_attn_store(a, tp, tokens, d_bad_id + 1, stream));
        RC(biased_attn_context(a, tp, tokens, max_new, plain_kernels, stream));
    }
    GatedRecurrence g = {};
    g.dtype = dtype;
    g.H = l.RH;
    g.dk = w.rk;
    g.dv = w.rv;
    g.q = at(buf.mix, w.col_rq);
    g.z = at(buf.mix, w.col_rf);
    g.v = at(buf.mix, w.col_rv);
    g.ld = w.n_mix;
    g.zb = w.zb;
    g.lower = w.lower;
    g.w = w.rnorm;
    g.eps = (float)c.eps;
    g.norm_width = l.rv;
    g.state = mem[i].state;
    g.out = at(buf.cat, w.cat_r);
    g.out_ld = w.n_cat;
    g.out_scale = (float)l.right_scale;
    g.work = buf.rec_work;
    RC(gated_recurrence(g, tp, tp.B, tokens, stream));
    pj = Projection{};
    pj.dtype = dtype;
    pj.M = tokens;
    pj.x = buf.cat;
    pj.W = w.w_out;
    pj.y = buf.x;
    pj.N = width;
    pj.K = w.n_cat;
    pj.f32 = 1;
    pj.resid = buf.x;
    return project(pj, stream);
}

// Final norm and head of some rows of the stream; logits in float, [n_rows, vocab].
int Finuvik::lm_head(float* stream_rows, const int* rows, int n_rows, void* hn, float* padded, float* out)
{
    RC(norm(stream_rows, rows, n_rows, final_norm, nullptr, hn, nullptr));
    Projection pj;
    pj.dtype = dtype;
    pj.M = n_rows;
    pj.x = hn;
    pj.W = head;
    pj.y = padded ? padded : out;
    pj.N = vocab_p;
    pj.K = width;
    pj.f32 = 1;
    RC(project(pj, stream));
    if (padded)
        ONELLM_CUDA(cudaMemcpy2DAsync(out, (size_t)c.vocab * sizeof(float), padded, (size_t)vocab_p * sizeof(float), (size_t)c.vocab * sizeof(float),
                                      n_rows, cudaMemcpyDeviceToDevice, stream));
    return ONELLM_OK;
}

int Finuvik::decode_layers(int step_bound, bool with_head)
{
    const TokenPositions tp = {nullptr, nullptr, batch, d_step, d_step_off};
    RC(embedding_pos_launch(dtype, d_ids, x, embed, pos, batch, width, c.vocab, max_seq_len, tp, d_bad_id, stream));
    const Buffers buf = {x, h1, h2, mix, cat, nullptr};
    for (size_t i = 0; i < c.layers.size(); i++) RC(layer(i, buf, batch, tp, 1, step_bound));
    return with_head ? lm_head(x, nullptr, batch, h1, logits_p, static_cast<float*>(logits)) : ONELLM_OK;
}

int Finuvik::context_layers(const ContextBatch& cb)
{
    const size_t T = cb.T, es = esize(), W = width;
    Carver cv{nullptr};
    Buffers buf = {};
    void* hn = nullptr;
    float* padded = nullptr;
    for (int pass = 0; pass < 2; pass++) {
        buf.x = cv.take<float>(T * W);
        buf.h1 = cv.take_bytes(T * W * es);
        buf.h2 = cv.take_bytes(T * W * es);
        buf.mix = cv.take_bytes(T * max_mix * es);
        buf.cat = cv.take_bytes(T * max_cat * es);
        size_t work = 0;
        for (size_t i = 0; i < c.layers.size(); i++)
            work = std::max(work, gated_recurrence_workspace(ONELLM_GR_TIED, (int)T, c.layers[i].RH, weights[i].rk, weights[i].rv));
        buf.rec_work = cv.take_bytes(work);
        hn = cv.take_bytes((size_t)cb.n_rows * W * es);
        padded = vocab_p == c.vocab ? nullptr : cv.take<float>((size_t)cb.n_rows * vocab_p);
        if (pass == 0) {
            RC(ensure_scratch(align_up(cv.off, 256)));
            cv = Carver{scratch};
        }
    }
    const TokenPositions tp = {cb.cu, cb.hist, cb.B, nullptr, nullptr};
    RC(embedding_pos_launch(dtype, d_prompt, buf.x, embed, pos, (int)T, width, c.vocab, max_seq_len, tp, d_bad_id, stream));
    for (size_t i = 0; i < c.layers.size(); i++) RC(layer(i, buf, (int)T, tp, cb.P, 0));
    RC(lm_head(buf.x, cb.rows, cb.n_rows, hn, padded, static_cast<float*>(cb.logits)));
    ONELLM_CHECK_LAUNCH();
    return ONELLM_OK;
}

// ---- weights -----------------------------------------------------------------------------------------------
int Finuvik::load(const std::string& folder)
{
    WeightPlacer f(dtype, stream);
    RC(f.file.open(folder + "/model.safetensors"));
    const int D = c.width;
    // plain [rows, width] tables keep their orientation
    RC(f.place("embed", embed, width, 0, 0, c.vocab, c.vocab, c.vocab, D, D, D, false));
    RC(f.place("pos", pos, width, 0, 0, c.max_positions, c.max_positions, c.max_positions, D, D, D, false));
    RC(f.place("head", head, vocab_p, 0, 0, c.vocab, c.vocab, c.vocab, D, D, D));
    RC(f.vec("final.norm", final_norm, D, D, D));
    for (size_t i = 0; i < c.layers.size(); i++) {
        if (!own(i)) continue;
        const FinuvikLayerConfig& l = c.layers[i];
        const FinuvikWeights& w = weights[i];
        const std::string p = "l" + std::to_string(i) + ".", a = p + "mix.left.", r = p + "mix.right.";
        RC(f.vec(p + "norm1", w.norm1, D, D, D));
        if (l.ff || f.file.find(p + "norm2")) RC(f.vec(p + "norm2", w.norm2, D, D, D));
        RC(f.place(a + "q", w.w_mix, w.n_mix, 0, 0, l.H * l.dk, l.dk, w.dk, D, D, D));
        RC(f.place(a + "k", w.w_mix, w.n_mix, 0, w.col_k, l.G * l.dk, l.dk, w.dk, D, D, D));
        RC(f.place(a + "v", w.w_mix, w.n_mix, 0, w.col_v, l.G * l.dv, l.dv, w.dv, D, D, D));
        RC(f.vec(a + "r1", w.r1, l.H, l.H, l.H));
        RC(f.vec(a + "r2", w.r2, l.H, l.H, l.H));
        RC(f.place(a + "o", w.w_out, width, 0, 0, D, D, D, l.H * l.dv, l.dv, w.dv));
        RC(f.place(r + "q", w.w_mix, w.n_mix, 0, w.col_rq, l.RH * l.rk, l.rk, w.rk, D, D, D));
        RC(f.place(r + "f", w.w_mix, w.n_mix, 0, w.col_rf, l.RH * l.rk, l.rk, w.rk, D, D, D));
        RC(f.place(r + "v", w.w_mix, w.n_mix, 0, w.col_rv, l.RH * l.rv, l.rv, w.rv, D, D, D));
        RC(f.vec(r + "f.b", w.zb, l.RH * l.rk, l.rk, w.rk));
        RC(f.vec(r + "lower", w.lower, l.RH * l.rk, l.rk, w.rk));
        RC(f.vec(r + "norm", w.rnorm, l.rv, l.rv, l.rv));
        RC(f.place(r + "o", w.w_out, width, w.cat_r, 0, D, D, D, l.RH * l.rv, l.rv, w.rv));
        if (l.ff) {
            RC(f.place(p + "mlp.gate", w.w_gate, w.ff, 0, 0, l.ff, l.ff, l.ff, D, D, D));
            RC(f.place(p + "mlp.up", w.w_up, w.ff, 0, 0, l.ff, l.ff, l.ff, D, D, D));
            RC(f.place(p + "mlp.down", w.w_out, width, w.cat_f, 0, D, D, D, l.ff, l.ff, l.ff));
        }
    }
    return finalize();
}

// What is computed from the weights once: the score tables of every layer with tensors of its own.
int Finuvik::finalize()
{
    for (size_t i = 0; i < c.layers.size(); i++) {
        if (!own(i)) continue;
        const FinuvikLayerConfig& l = c.layers[i];
        const FinuvikWeights& w = weights[i];
        RC(build_query_factor(w.q_factor, max_seq_len, l.scale, l.temp_coef, l.temp_every, stream));
        RC(build_distance_penalty(w.penalty, w.r1, w.r2, l.H, max_seq_len, stream));
    }
    ONELLM_CUDA(cudaStreamSynchronize(stream));
    weights_ready = true;
    return ONELLM_OK;
}

// Random weights of the configured shape (padding included: sizes are then what the kernels see), gates that forget
// slowly and a mild distance penalty.
int Finuvik::init_random(uint64_t seed, float std)
{
    auto normal = [&](void* w, size_t rows, size_t cols, uint64_t tag) { return init_normal(dtype, w, rows, cols, cols, 0, 0, seed, tag, 0.f, std, stream); };
    auto fill = [&](float* w, size_t n, float v) { return init_normal(ONELLM_F32, w, 1, n, n, 0, 0, seed, 7, v, 0.f, stream); };
    for (size_t i = 0; i < c.layers.size(); i++) {
        if (!own(i)) continue;
        const FinuvikLayerConfig& l = c.layers[i];
        const FinuvikWeights& w = weights[i];
        const uint64_t t0 = 16 * (uint64_t)i + 32;
        RC(normal(w.w_mix, width, w.n_mix, t0));
        if (w.ff) {
            RC(normal(w.w_gate, width, w.ff, t0 + 1));
            RC(normal(w.w_up, width, w.ff, t0 + 2));
        }
        RC(normal(w.w_out, w.n_cat, width, t0 + 3));
        RC(fill(w.r1, l.H, 1.0f));
        RC(fill(w.r2, l.H, 0.1f));
        RC(fill(w.zb, (size_t)l.RH * w.rk, 2.0f));
        RC(fill(w.lower, (size_t)l.RH * w.rk, 0.5f));
        RC(fill(w.rnorm, w.rv, 1.0f));
        RC(fill(w.norm1, width, 0.0f));
        RC(fill(w.norm2, width, 0.0f));
    }
    RC(normal(embed, c.vocab, width, 1000001));
    RC(normal(pos, c.max_positions, width, 1000003));
    RC(normal(head, width, vocab_p, 1000002));
    RC(fill(final_norm, width, 0.0f));
    return finalize();
}

static int make_finuvik(const Json& config, const std::string& folder, const ModelOptions& opt, Engine** out)
{
    Finuvik* m = new Finuvik();
    int rc = read_config(config, &m->c);
    if (!rc) {
        m->dtype = opt.dtype;
        m->vocab = m->c.vocab;
        m->width = pad_to(m->c.width, 16);
        m->vocab_p = pad_to(m->c.vocab, 8);
        m->logits_dtype = ONELLM_F32;
        m->eos_id = -1;  // the design names no end-of-sequence token
        m->max_batch = opt.max_batch;
        m->max_seq_len = opt.max_seq_len > 0 ? std::min(opt.max_seq_len, m->c.max_positions) : m->c.max_positions;
        if (opt.max_batch < 1 || opt.max_batch > 64) {
            set_error("model_open: max_batch %d outside [1, 64]", opt.max_batch);
            rc = ONELLM_ERR_ARG;
        }
    }
    if (!rc) rc = m->allocate();  // the arena starts as zeros: so do the padding of the weights, the caches and the states
    if (!rc && !folder.empty()) rc = m->load(folder);
    if (rc) {
        delete m;
        return rc;
    }
    *out = m;
    return ONELLM_OK;
}

static const ModelRegistration register_finuvik("Finuvik", make_finuvik);

}  // namespace onellm
