// Lenolix for the decode driver: layers of grouped-query attention (a window, kept first tokens, sinks, halves rotated with stretched
// wavelengths) and gated feed-forwards with clamped halves, layer norms on both sides of every sublayer, embeddings of token pairs, and a
// stretch of layers that runs several times, each pass entered through a mat-mul over the stream and the embedding output.
//
// A step's graph keeps the residual stream in F32.  q, k and v weights are one device matrix, the rows of gate and up weights alternate
// in another (the mat-mul's epilogue takes a pair), and the entry of a pass is split by columns: the part that reads the embedding
// output is the same in every pass and runs once.  A sublayer's output norm, channel scale, residual sum and the norm of what follows
// are one node, so a layer is seven launches while rows are few (eight in a prompt).
#include "arch_dense.h"

namespace b200 {
namespace {

constexpr int64_t ATTN_FEW = 8;              // rows per sequence up to which attention runs row by row over the cells
constexpr int64_t SPLIT_KEYS = 32, SPLIT_MAX = 8, SPLIT_CTAS = 592;   // keys a block takes at least, blocks of a row's cluster, blocks wanted
constexpr float GATE_ALPHA = 1.702f;

struct Layer {
    int64_t heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int64_t window = 0, keep = 0;            // window 0: no mask
    float scale = 1.0f;
    int64_t rot_dims = 0;
    float rot_base = 1.0f, rot_factor = 0.0f, rot_low = 0.0f, rot_high = 0.0f, rot_original = 0.0f;   // factor 0: no scaling
    int64_t ff = 0;                          // 0: no feed-forward
    float limit = 0.0f;
    int64_t q_rows() const { return heads * dim; }
    int64_t k_rows() const { return kv_heads * dim; }
    int64_t v_rows() const { return kv_heads * vdim; }
    int64_t proj_rows() const { return q_rows() + k_rows() + v_rows(); }
    int64_t cell_row() const { return kv_heads * ((dim + 7) / 8 * 8 + (vdim + 7) / 8 * 8); }   // elements of a cell's row
};

class LenolixArch : public Arch {
public:
    int dtype = B200_TYPE_BF16;
    int64_t vocab = 0, width = 0;
    float eps = 1e-5f, embed_scale = 1.0f;
    int64_t buckets = 0, mul_prev = 0, mul_cur = 0;   // buckets 0: no table of pairs
    std::vector<Layer> layers;
    LoopSpec loop;

    const char *name() const override { return "Lenolix"; }
    int32_t n_vocab() const override { return (int32_t)vocab; }
    bool masked_cache() const override { return false; }
    int64_t key_span() const override {
        int64_t span = 1;
        for (const Layer &l : layers) {
            if (l.window == 0) return 0;
            span = std::max(span, l.window);
        }
        return span;
    }
    int64_t kept_first() const override {
        int64_t keep = 0;
        for (const Layer &l : layers) keep = std::max(keep, l.keep);
        return keep;
    }
    std::vector<std::pair<int64_t, int64_t>> runs() const { return layer_runs((int64_t)layers.size(), loop); }

    // per layer run: its cells' rows
    int alloc_memory(b200_llama *c) override {
        const auto rs = runs();
        c->mem_l.resize(rs.size());
        std::vector<size_t> at(rs.size());
        size_t bytes = 0;
        for (size_t i = 0; i < rs.size(); i++) {
            init_tensor(&c->mem_l[i], dtype, layers[rs[i].first].cell_row(), c->n_ctx);
            snprintf(c->mem_l[i].name, sizeof(c->mem_l[i].name), "cells_r%zu", i);
            at[i] = bytes;
            bytes += (c->mem_l[i].nb[2] + TENSOR_ALIGN - 1) / TENSOR_ALIGN * TENSOR_ALIGN;
        }
        c->kv_buf = c->buft->iface.alloc_buffer(c->buft, std::max<size_t>(bytes, TENSOR_ALIGN));
        if (!c->kv_buf) return B200_STATUS_ALLOC_FAILED;
        c->kv_buf->iface.clear(c->kv_buf, 0);   // (the padding of a cell's row stays zero)
        uint8_t *b = (uint8_t *)c->kv_buf->iface.get_base(c->kv_buf);
        for (size_t i = 0; i < rs.size(); i++) {
            c->mem_l[i].buffer = c->kv_buf;
            c->mem_l[i].data = b + at[i];
        }
        return B200_STATUS_SUCCESS;
    }

    std::vector<StepShape> largest(const b200_llama *c) const override {
        std::vector<StepShape> v;
        for (int64_t n : {(int64_t)c->n_batch, std::min<int64_t>(c->n_batch, FEW_ROWS)}) {
            StepShape s;
            s.n = s.n_out = s.max_rows = n;
            s.n_seg = std::min<int64_t>(n, c->n_seq);
            s.n_tab = s.max_keys = (c->n_ctx + KV_PAD - 1) / KV_PAD * KV_PAD;
            v.push_back(s);
        }
        return v;
    }

    bool place(const std::string &t, TensorPlace *p) const override {
        const auto matrix = [&](const std::string &dst, int64_t k, int64_t n, int64_t row0, int64_t rows, int64_t step = 1) {
            p->dst = dst; p->type = dtype; p->ne0 = k; p->ne1 = n; p->row0 = row0; p->rows = rows; p->row_step = step; p->plus_one = false;
            return true;
        };
        const auto vec = [&](int64_t n, int64_t rows = 1) {
            p->dst = t; p->type = B200_TYPE_F32; p->ne0 = n; p->ne1 = rows; p->row0 = 0; p->rows = rows; p->row_step = 1; p->plus_one = false;
            return true;
        };
        if (t == "embed") return matrix(t, width, vocab, 0, vocab);
        if (t == "bigram" && buckets > 0) return matrix(t, width, buckets + 1, 0, buckets + 1);
        if (t == "final.norm" || t == "final.norm.b") return vec(width);
        if (loop.times > 0 && t == "loop.in") return matrix(t, 2 * width, width, 0, width);
        if (loop.times > 0 && t == "loop.step") return vec(width, loop.times);
        int64_t il = 0;
        std::string pre, rest;
        if (!split_layer_name(t, (int64_t)layers.size(), &il, &pre, &rest)) return false;
        const Layer &l = layers[il];
        for (const char *n : {"norm1", "norm1b", "norm2", "norm2b"})
            if (rest == n || rest == std::string(n) + ".b") return vec(width);
        if (rest == "ls1" || rest == "ls2") return vec(width);
        const std::string proj = pre + "mix.proj", pairs = pre + "mlp.pairs";
        if (rest == "mix.q") return matrix(proj, width, l.proj_rows(), 0, l.q_rows());
        if (rest == "mix.k") return matrix(proj, width, l.proj_rows(), l.q_rows(), l.k_rows());
        if (rest == "mix.v") return matrix(proj, width, l.proj_rows(), l.q_rows() + l.k_rows(), l.v_rows());
        if (rest == "mix.sink") return vec(l.heads);
        if (rest == "mix.o") return matrix(t, l.heads * l.vdim, width, 0, width);
        if (l.ff > 0) {
            if (rest == "mlp.gate") return matrix(pairs, width, 2 * l.ff, 0, l.ff, 2);
            if (rest == "mlp.up") return matrix(pairs, width, 2 * l.ff, 1, l.ff, 2);
            if (rest == "mlp.down") return matrix(t, l.ff, width, 0, width);
        }
        return false;
    }
    std::vector<std::string> tensor_names() const override {
        std::vector<std::string> v = {"embed", "final.norm", "final.norm.b"};
        if (buckets > 0) v.push_back("bigram");
        if (loop.times > 0) v.insert(v.end(), {"loop.in", "loop.step"});
        for (size_t i = 0; i < layers.size(); i++) {
            const std::string p = "l" + std::to_string(i) + ".";
            const auto add = [&](std::initializer_list<const char *> names) { for (const char *n : names) v.push_back(p + n); };
            add({"norm1", "norm1.b", "norm1b", "norm1b.b", "ls1", "mix.q", "mix.k", "mix.v", "mix.sink", "mix.o"});
            if (layers[i].ff > 0) add({"norm2", "norm2.b", "norm2b", "norm2b.b", "ls2", "mlp.gate", "mlp.up", "mlp.down"});
        }
        return v;
    }

    int build(b200_llama *c, Graph *g, uint8_t *base, const StepShape &s) override;
};

int LenolixArch::build(b200_llama *c, Graph *g, uint8_t *base, const StepShape &s) {
    int rc = require_tensors(c, *this);
    if (rc != B200_STATUS_SUCCESS) return rc;
    const int64_t n = s.n, E = width;
    StepBuilder b;
    b.c = c;
    b.g = g;
    b.base = base;
    b.few = n <= FEW_ROWS;
    b.act = dtype == B200_TYPE_F32 || b.few ? B200_TYPE_F32 : B200_TYPE_BF16;
    b.eps = eps;
    b.inputs(s);
    ggml_tensor *resid[2] = {b.alloc(B200_TYPE_F32, E, n, 1, "resid_a"), b.alloc(B200_TYPE_F32, E, n, 1, "resid_b")};
    ggml_tensor *rows = b.alloc(b.act, E, n, 1, "rows");   // what the next mat-mul reads
    int side = 0;
    const auto next_slot = [&]() { return resid[side ^= 1]; };
    const auto W = [&](const std::string &name) { return weight(c, name); };
    const bool copies = b.act != B200_TYPE_F32;            // the stream's own type is not what mat-muls read

    ggml_tensor *x = b.op(b.over(resid[side], "inp_embd"), B200_OP_PAIR_EMBED, W("embed"), g->tokens);
    x->op_params[0] = bits(embed_scale);
    if (buckets > 0) {
        g->prev = b.alloc(B200_TYPE_I32, n, 1, 1, "inp_prev");
        x->src[2] = g->prev;
        x->src[3] = W("bigram");
        x->op_params[1] = (int32_t)(mul_prev % buckets);
        x->op_params[2] = (int32_t)(mul_cur % buckets);
    }
    ggml_tensor *stream = x;                               // the stream in the type mat-muls read, where a pass wants it
    ggml_tensor *enter_x = nullptr, *from_embd = nullptr;  // the pass entry's weight on the stream; its other half's result
    if (loop.times > 0) {
        ggml_tensor *in = W("loop.in");
        enter_x = b.view_2d(in, E, E, in->nb[1], 0);
        ggml_tensor *enter_0 = b.view_2d(in, E, E, in->nb[1], (size_t)E * in->nb[0]);
        if (copies) x->src[4] = stream = b.alloc(b.act, E, n, 1, "stream_rows");
        from_embd = b.dense(b.alloc(B200_TYPE_F32, E, n, 1, "from_embd"), enter_0, stream, nullptr, nullptr, ACT_NONE);
    }
    const size_t layer_base = b.off;
    const auto rs = runs();
    const auto begins = [&](size_t r) { return r < rs.size() && rs[r].second >= 0 && rs[r].first == loop.start; };
    ggml_tensor *h = nullptr;                              // the normed rows of the coming sublayer, if a node has made them
    // the residual sum behind a sublayer and the rows of what follows: the norm `next` of a coming sublayer, or a pass's input
    const auto close = [&](ggml_tensor *y, const std::string &p, const std::string &which, const std::string &next, bool pass, const char *name) {
        ggml_tensor *t = b.op(b.over(next_slot(), name), B200_OP_NORM_SUM, x, y, W(p + "norm" + which + "b"), W(p + "norm" + which + "b.b"));
        t->src[4] = W(p + "ls" + which);
        t->op_params[0] = bits(eps);
        h = nullptr;
        stream = t;
        if (!next.empty()) {
            t->src[5] = W(next);
            t->src[6] = W(next + ".b");
            t->src[7] = h = rows;
        } else if (pass && copies) {
            t->src[7] = stream = rows;
        }
        x = t;
    };
    for (size_t r = 0; r < rs.size(); r++) {
        b.off = layer_base;
        const Layer &l = layers[rs[r].first];
        const std::string p = "l" + std::to_string(rs[r].first) + ".";
        if (begins(r)) {
            ggml_tensor *steps = W("loop.step"), *step = b.view_2d(steps, E, 1, steps->nb[1], (size_t)rs[r].second * steps->nb[1]);
            x = b.dense(b.over(next_slot(), "pass_in"), enter_x, stream, from_embd, nullptr, ACT_NONE);
            x->src[4] = step;
            h = nullptr;
        }
        if (!h) {
            h = b.op(b.over(rows, "norm_rows"), B200_OP_LAYER_NORM_W, x, W(p + "norm1"), W(p + "norm1.b"));
            h->op_params[0] = bits(eps);
        }
        const std::string follows = r + 1 < rs.size() && !begins(r + 1) ? "l" + std::to_string(rs[r + 1].first) + ".norm1" : "";
        ggml_tensor *proj = b.dense(b.alloc(B200_TYPE_F32, l.proj_rows(), n, 1, "proj"), W(p + "mix.proj"), h, nullptr, nullptr, ACT_NONE);
        const bool few = s.max_rows <= ATTN_FEW;
        const int64_t rep = l.heads / l.kv_heads, keys = l.window > 0 ? std::min(s.max_keys, l.window + l.keep) : s.max_keys;
        int64_t splits = 1;
        while (splits < SPLIT_MAX && 2 * splits * SPLIT_KEYS <= keys && 2 * splits * n * l.kv_heads * ((rep + 7) / 8) <= SPLIT_CTAS) splits *= 2;
        const int32_t prm[14] = {(int32_t)l.heads, (int32_t)l.kv_heads, (int32_t)l.dim, (int32_t)l.vdim, (int32_t)l.window, (int32_t)l.keep, bits(l.scale), (int32_t)l.rot_dims,
                                 bits(l.rot_base), bits(l.rot_factor), bits(l.rot_low), bits(l.rot_high), bits(l.rot_original), (int32_t)splits};
        ggml_tensor *cache = &c->mem_l[r];
        if (!few) {
            ggml_tensor *st = b.op(b.alias_of(cache), B200_OP_GROUPED_STORE, proj, g->pos, g->cells);
            memcpy(st->op_params, prm, sizeof(prm));
        }
        ggml_tensor *mixed = b.op(b.alloc(b.act, l.heads * l.vdim, n, 1, "attn_out"), few ? B200_OP_GROUPED_DECODE : B200_OP_GROUPED_ATTN, proj, g->pos, g->cells, cache);
        mixed->src[4] = g->row_seg;
        mixed->src[5] = g->seg;
        mixed->src[6] = g->tab;
        mixed->src[7] = W(p + "mix.sink");
        memcpy(mixed->op_params, prm, sizeof(prm));
        ggml_tensor *y = b.dense(b.alloc(B200_TYPE_F32, E, n, 1, "mix_out"), W(p + "mix.o"), mixed, nullptr, nullptr, ACT_NONE);
        close(y, p, "1", l.ff > 0 ? p + "norm2" : follows, begins(r + 1), "mix_sum");
        if (l.ff > 0) {
            ggml_tensor *ff = b.dense(b.alloc(b.act, l.ff, n, 1, "ff_rows"), W(p + "mlp.pairs"), h, nullptr, nullptr, ACT_CLAMPED_GATE);
            ff->op_params[2] = bits(l.limit);
            ff->op_params[3] = bits(GATE_ALPHA);
            y = b.dense(b.alloc(B200_TYPE_F32, E, n, 1, "ff_out"), W(p + "mlp.down"), ff, nullptr, nullptr, ACT_NONE);
            close(y, p, "2", follows, begins(r + 1), "l_out");
        }
    }
    b.off = layer_base;
    x = b.get_rows(x, g->out_ids, "result_rows");
    const int out_act = dtype == B200_TYPE_F32 || s.n_out <= FEW_ROWS ? B200_TYPE_F32 : B200_TYPE_BF16;
    x = b.layer_norm(out_act, x, W("final.norm"), W("final.norm.b"), "result_norm");
    g->logits = b.dense(b.alloc(B200_TYPE_F32, vocab, s.n_out, 1, "result_output"), W("embed"), x, nullptr, nullptr, ACT_NONE);
    g->argmax = b.op(b.alloc(B200_TYPE_I32, s.n_out, 1, 1, "argmax"), GGML_OP_ARGMAX, g->logits);
    g->bytes = b.high;
    return B200_STATUS_SUCCESS;
}

}  // namespace

std::unique_ptr<Arch> lenolix_from_config(const Json &config, int dtype, std::string *err) {
    std::unique_ptr<LenolixArch> a(new LenolixArch());
    Field f{err};
    const auto there = [](const Json *j) { return j && !j->is_null(); };
    const auto fail = [&](const char *m) {
        if (err->empty()) *err = std::string("config: ") + m;
    };
    a->dtype = dtype;
    a->vocab = f.size(config, "vocab", "model");
    a->width = f.size(config, "width", "model");
    if (const Json *norm = f.get(config, "norm", "model")) a->eps = (float)f.number(*norm, "eps", "norm");
    const Json *emb = config.find("embedding");
    if (there(emb)) {
        if (emb->find("scale")) a->embed_scale = (float)f.number(*emb, "scale", "embedding");
        const Json *pairs = emb->find("bigram");
        if (there(pairs)) {
            a->buckets = f.size(*pairs, "buckets", "bigram");
            const double prev = f.number(*pairs, "mul_prev", "bigram"), cur = f.number(*pairs, "mul_cur", "bigram");
            if (prev != std::floor(prev) || cur != std::floor(cur) || prev < 0 || cur < 0 || prev > 9e15 || cur > 9e15) fail("the bigram factors are not usable integers");
            a->mul_prev = (int64_t)prev;
            a->mul_cur = (int64_t)cur;
        }
    }
    const Json *layers = f.get(config, "layers", "model");
    if (layers && layers->items.empty()) fail("no layers");
    for (const Json &j : layers ? layers->items : std::vector<Json>()) {
        Layer l;
        const Json *type = f.get(j, "type", "layer"), *mix = f.get(j, "mixer", "layer");
        if (!type || !mix) break;
        if (type->str != "attention" && err->empty()) *err = "config: layer type '" + type->str + "' is not known";
        l.heads = f.size(*mix, "heads", "mixer");
        l.kv_heads = f.size(*mix, "kv_heads", "mixer");
        l.dim = f.size(*mix, "dim", "mixer");
        l.vdim = f.size(*mix, "vdim", "mixer");
        l.scale = (float)f.number(*mix, "scale", "mixer");
        if (!err->empty()) break;
        if (l.heads % l.kv_heads) fail("heads must be a multiple of kv_heads");
        const Json *mask = mix->find("mask");
        if (there(mask)) {
            l.window = f.size(*mask, "size", "mask");
            if (mask->find("keep_first")) l.keep = f.size(*mask, "keep_first", "mask", 0);
        }
        const Json *rot = mix->find("rot");
        if (there(rot)) {
            l.rot_dims = f.size(*rot, "dims", "rot", 0);
            l.rot_base = (float)f.number(*rot, "base", "rot");
            if (l.rot_dims % 2 || l.rot_dims > l.dim) fail("rotated dimensions must be an even part of dim");
            const Json *sc = rot->find("scaling");
            if (there(sc)) {
                l.rot_factor = (float)f.number(*sc, "factor", "scaling");
                l.rot_low = (float)f.number(*sc, "low", "scaling");
                l.rot_high = (float)f.number(*sc, "high", "scaling");
                l.rot_original = (float)f.number(*sc, "original", "scaling");
                if (!(l.rot_factor > 0.0f && l.rot_low > 0.0f && l.rot_high >= l.rot_low && l.rot_original > 0.0f)) fail("the rotary scaling is not usable");
            }
        }
        const Json *mlp = j.find("mlp");
        if (there(mlp)) {
            const Json *kind = mlp->find("kind");
            if (!kind || kind->str != "dense") fail("only dense feed-forwards are known");
            l.ff = f.size(*mlp, "ff", "mlp");
            l.limit = (float)f.number(*mlp, "limit", "mlp");
        }
        a->layers.push_back(l);
    }
    a->loop = f.loop(config, (int64_t)a->layers.size());
    if (!err->empty()) return nullptr;
    return a;
}

}  // namespace b200
