// Rukusun for the decode driver: layers of gated linear attention and of latent attention in any order, each with an optional
// dense feed-forward, a stretch of layers that can run several times, everything by configuration.
//
// A step's graph keeps the residual stream in F32.  Weights that read the same rows are one device matrix (q, k, v, gate and
// decay input of a linear-attention layer; query, latent and gate of a latent-attention layer; key and value weights of the
// latent), so a layer is a handful of nodes.  Two forms of a step: few rows keep every activation in F32 and run the norms
// inside the mat-muls; many rows (BF16 models) hand the mat-muls BF16 rows.  Attention over the latents has two forms as well:
// queries taken through the key weight, against the cached latents themselves (a few rows per sequence), or keys and values
// expanded from the latents for the positions the step can see (a prompt's rows).
#include "arch_dense.h"

namespace b200 {
namespace {

constexpr int64_t GLA_TOKENWISE = 16;      // rows per sequence up to which the recurrence runs token by token
constexpr int64_t LATENT_FEW = 8;          // rows per sequence up to which attention reads the latents themselves
constexpr int64_t SPLIT_KEYS = 32;         // keys a split of that attention is cut into
constexpr int64_t SPLIT_CTAS = 296, SPLIT_HEADS = 8;

enum LayerType { GLA, LATENT };
struct Layer {
    LayerType type = GLA;
    int64_t heads = 0, dim = 0, vdim = 0;
    float tau = 1.0f;
    int64_t decay_rank = 0;                // known once the tensor's shape is
    int64_t kv_rank = 0, rot = 0, rot_dims = 0, window = 0;
    float scale = 1.0f, rot_base = 10000.0f;
    int64_t ff = 0;                        // 0: no feed-forward
    int64_t cell_row() const { return (kv_rank + rot + 7) / 8 * 8; }   // elements of a cell's row
};

class RukusunArch : public Arch {
public:
    int dtype = B200_TYPE_BF16;
    int64_t vocab = 0, width = 0;
    float eps = 1e-5f, embed_scale = 1.0f;
    std::vector<Layer> layers;
    LoopSpec loop;

    const char *name() const override { return "Rukusun"; }
    int32_t n_vocab() const override { return (int32_t)vocab; }
    bool masked_cache() const override { return false; }
    int64_t key_span() const override {
        int64_t span = -1;
        for (const Layer &l : layers) {
            if (l.type != LATENT) continue;
            if (l.window == 0) return 0;
            span = std::max(span, l.window);
        }
        return span;
    }
    std::vector<std::pair<int64_t, int64_t>> runs() const { return layer_runs((int64_t)layers.size(), loop); }

    // per layer run: the cell rows of a latent-attention layer, the state slots of a linear-attention layer
    int alloc_memory(b200_llama *c) override {
        const auto rs = runs();
        c->mem_l.resize(rs.size());
        std::vector<size_t> at(rs.size());
        size_t bytes = 0;
        for (size_t i = 0; i < rs.size(); i++) {
            const Layer &l = layers[rs[i].first];
            if (l.type == GLA) init_tensor(&c->mem_l[i], B200_TYPE_F32, l.heads * l.dim * l.vdim, c->n_seq);
            else init_tensor(&c->mem_l[i], dtype, l.cell_row(), c->n_ctx);
            snprintf(c->mem_l[i].name, sizeof(c->mem_l[i].name), "%s_r%zu", l.type == GLA ? "state" : "cells", i);
            at[i] = bytes;
            bytes += (c->mem_l[i].nb[2] + TENSOR_ALIGN - 1) / TENSOR_ALIGN * TENSOR_ALIGN;
        }
        c->kv_buf = c->buft->iface.alloc_buffer(c->buft, std::max<size_t>(bytes, TENSOR_ALIGN));
        if (!c->kv_buf) return B200_STATUS_ALLOC_FAILED;
        c->kv_buf->iface.clear(c->kv_buf, 0);
        uint8_t *b = (uint8_t *)c->kv_buf->iface.get_base(c->kv_buf);
        for (size_t i = 0; i < rs.size(); i++) {
            c->mem_l[i].buffer = c->kv_buf;
            c->mem_l[i].data = b + at[i];
        }
        return B200_STATUS_SUCCESS;
    }

    std::vector<StepShape> largest(const b200_llama *c) const override {
        std::vector<StepShape> v;
        for (int64_t n : {(int64_t)c->n_batch, std::min<int64_t>(c->n_batch, FEW_ROWS)})
            for (int64_t rows : {(int64_t)1, n}) {
                StepShape s;
                s.n = s.n_out = rows == 1 ? std::min<int64_t>(n, c->n_seq * LATENT_FEW) : n;
                s.n_seg = std::min<int64_t>(n, c->n_seq);
                const int64_t all = (c->n_ctx + KV_PAD - 1) / KV_PAD * KV_PAD;
                s.n_tab = all;
                s.max_keys = all;
                s.max_rows = rows;
                v.push_back(s);
            }
        return v;
    }

    bool place(const std::string &t, TensorPlace *p) const override {
        const auto matrix = [&](const std::string &dst, int64_t k, int64_t n, int64_t row0, int64_t rows) {
            p->dst = dst; p->type = dtype; p->ne0 = k; p->ne1 = n; p->row0 = row0; p->rows = rows; p->plus_one = false;
            return true;
        };
        const auto vec = [&](int64_t n, bool plus_one, int64_t rows = 1) {
            p->dst = t; p->type = B200_TYPE_F32; p->ne0 = n; p->ne1 = rows; p->row0 = 0; p->rows = rows; p->plus_one = plus_one;
            return true;
        };
        if (t == "embed" || t == "head") return matrix(t, width, vocab, 0, vocab);
        if (t == "final.norm") return vec(width, true);
        if (t == "loop.step" && loop.times > 0) return vec(width, false, loop.times);
        int64_t il = 0;
        std::string pre, rest;
        if (!split_layer_name(t, (int64_t)layers.size(), &il, &pre, &rest)) return false;
        const Layer &l = layers[il];
        if (rest == "norm1") return vec(width, true);
        if (l.ff > 0) {
            if (rest == "norm2") return vec(width, true);
            if (rest == "mlp.up") return matrix(t, width, l.ff, 0, l.ff);
            if (rest == "mlp.down") return matrix(t, l.ff, width, 0, width);
        }
        if (l.type == GLA) {
            const int64_t d = l.heads * l.dim, e = l.heads * l.vdim, n = proj_rows(l);
            if (rest == "mix.q") return matrix(pre + "mix.proj", width, n, 0, d);
            if (rest == "mix.k") return matrix(pre + "mix.proj", width, n, d, d);
            if (rest == "mix.v") return matrix(pre + "mix.proj", width, n, 2 * d, e);
            if (rest == "mix.g") return matrix(pre + "mix.proj", width, n, 2 * d + e, e);
            if (rest == "mix.a1") return matrix(pre + "mix.proj", width, n, 2 * d + 2 * e, l.decay_rank);
            if (rest == "mix.a2") return matrix(t, l.decay_rank, d, 0, d);
            if (rest == "mix.a2.b") return vec(d, false);
            if (rest == "mix.norm") return vec(l.vdim, false);
            if (rest == "mix.o") return matrix(t, e, width, 0, width);
        } else {
            const int64_t q = l.heads * (l.dim + l.rot), n = proj_rows(l);
            if (rest == "mix.q") return matrix(pre + "mix.proj", width, n, 0, q);
            if (rest == "mix.dkv") return matrix(pre + "mix.proj", width, n, q, l.kv_rank + l.rot);
            if (rest == "mix.g") return matrix(pre + "mix.proj", width, n, q + l.kv_rank + l.rot, l.heads);
            if (rest == "mix.dkv.norm") return vec(l.kv_rank, false);
            if (rest == "mix.uk") return matrix(pre + "mix.ukv", l.kv_rank, l.heads * (l.dim + l.vdim), 0, l.heads * l.dim);
            if (rest == "mix.uv") return matrix(pre + "mix.ukv", l.kv_rank, l.heads * (l.dim + l.vdim), l.heads * l.dim, l.heads * l.vdim);
            if (rest == "mix.sink") return vec(l.heads, false);
            if (rest == "mix.o") return matrix(t, l.heads * l.vdim, width, 0, width);
        }
        return false;
    }
    std::vector<std::string> tensor_names() const override {
        std::vector<std::string> v = {"embed", "head", "final.norm"};
        if (loop.times > 0) v.push_back("loop.step");
        for (size_t i = 0; i < layers.size(); i++) {
            const std::string p = "l" + std::to_string(i) + ".";
            const auto add = [&](std::initializer_list<const char *> names) { for (const char *n : names) v.push_back(p + n); };
            add({"norm1"});
            if (layers[i].ff > 0) add({"norm2", "mlp.up", "mlp.down"});
            if (layers[i].type == GLA) add({"mix.q", "mix.k", "mix.v", "mix.g", "mix.a1", "mix.a2", "mix.a2.b", "mix.norm", "mix.o"});
            else add({"mix.q", "mix.dkv", "mix.dkv.norm", "mix.uk", "mix.uv", "mix.sink", "mix.g", "mix.o"});
        }
        return v;
    }
    // the rank of the decay's two weights is a tensor's shape, not a configured number
    bool learn_shape(const std::string &t, int64_t, int64_t ne1) override {
        const std::string tail = ".mix.a1";
        if (t.size() <= tail.size() || t.compare(t.size() - tail.size(), tail.size(), tail) != 0 || t[0] != 'l') return true;
        const size_t il = (size_t)atoll(t.c_str() + 1);
        if (il >= layers.size() || layers[il].type != GLA) return true;
        if (layers[il].decay_rank != 0 && layers[il].decay_rank != ne1) return false;
        layers[il].decay_rank = ne1;
        return true;
    }

    int build(b200_llama *c, Graph *g, uint8_t *base, const StepShape &s) override;

private:
    static int64_t proj_rows(const Layer &l) {
        if (l.type == GLA && l.decay_rank == 0) return 0;   // not known yet
        return l.type == GLA ? 2 * l.heads * l.dim + 2 * l.heads * l.vdim + l.decay_rank : l.heads * (l.dim + l.rot) + l.kv_rank + l.rot + l.heads;
    }
};

int RukusunArch::build(b200_llama *c, Graph *g, uint8_t *base, const StepShape &s) {
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
    int side = 0;
    const auto next_slot = [&]() { return resid[side ^= 1]; };
    const auto W = [&](const std::string &name) { return weight(c, name); };

    int rc = require_tensors(c, *this);
    if (rc != B200_STATUS_SUCCESS) return rc;

    ggml_tensor *x = b.take_rows(B200_TYPE_F32, W("embed"), g->tokens, embed_scale, resid[side], "inp_embd");
    const size_t layer_base = b.off;
    const auto rs = runs();
    for (size_t r = 0; r < rs.size(); r++) {
        b.off = layer_base;
        const Layer &l = layers[rs[r].first];
        const std::string p = "l" + std::to_string(rs[r].first) + ".";
        if (rs[r].second >= 0 && rs[r].first == loop.start) {
            ggml_tensor *steps = W("loop.step");
            ggml_tensor *row = b.view_2d(steps, E, 1, steps->nb[1], (size_t)rs[r].second * steps->nb[1]);
            x = b.op(b.over(next_slot(), "loop_step"), GGML_OP_ADD, x, row);
        }
        ggml_tensor *proj = b.normed_dense(W(p + "mix.proj"), x, W(p + "norm1"), B200_TYPE_F32, 0, "proj");
        ggml_tensor *mixed = nullptr;
        if (l.type == GLA) {
            const int64_t d = l.heads * l.dim, e = l.heads * l.vdim;
            ggml_tensor *scratch = nullptr;
            if (s.max_rows > GLA_TOKENWISE) {
                const size_t floats = gla_scratch_floats(l.heads, l.dim, l.vdim, n, s.n_seg);
                scratch = b.alloc(B200_TYPE_F32, (int64_t)floats, 1, 1, "gla_scratch");
            }
            mixed = b.op(b.alloc(b.act, e, n, 1, "gla_out"), B200_OP_GLA, proj, W(p + "mix.a2"), W(p + "mix.a2.b"), W(p + "mix.norm"));
            mixed->src[4] = &c->mem_l[r];
            mixed->src[5] = g->seg;
            mixed->src[6] = scratch;
            const int32_t prm[13] = {(int32_t)l.heads, (int32_t)l.dim, (int32_t)l.vdim, 0, (int32_t)d, (int32_t)(2 * d), (int32_t)(2 * d + e), (int32_t)(2 * d + 2 * e),
                                     bits(1.0f / sqrtf((float)l.dim)), bits(1.0f / l.tau), bits(eps), (int32_t)s.max_rows, (int32_t)l.decay_rank};
            memcpy(mixed->op_params, prm, sizeof(prm));
        } else {
            const int64_t q = l.heads * (l.dim + l.rot), R = l.kv_rank;
            ggml_tensor *cache = &c->mem_l[r], *ukv = W(p + "mix.ukv"), *cn = W(p + "mix.dkv.norm"), *sink = W(p + "mix.sink");
            int64_t keys = s.max_keys;
            if (l.window > 0) keys = std::min(keys, (l.window + SPLIT_KEYS - 1) / SPLIT_KEYS * SPLIT_KEYS);
            const int64_t groups = n * ((l.heads + SPLIT_HEADS - 1) / SPLIT_HEADS);
            int64_t splits = std::max<int64_t>(1, std::min((keys + SPLIT_KEYS - 1) / SPLIT_KEYS, SPLIT_CTAS / groups));
            const int64_t per = ((keys + splits - 1) / splits + SPLIT_KEYS - 1) / SPLIT_KEYS * SPLIT_KEYS;
            splits = (keys + per - 1) / per;
            const int32_t prm[15] = {(int32_t)l.heads, (int32_t)l.dim, (int32_t)l.rot, (int32_t)R, (int32_t)l.vdim, (int32_t)l.window, bits(l.scale), bits(eps),
                                     bits(l.rot_base), (int32_t)l.rot_dims, 0, (int32_t)q, (int32_t)(q + R + l.rot), (int32_t)per, (int32_t)splits};
            const auto set = [&](ggml_tensor *t) { memcpy(t->op_params, prm, sizeof(prm)); return t; };
            if (s.max_rows <= LATENT_FEW) {
                ggml_tensor *ql = set(b.op(b.alloc(B200_TYPE_F32, R + l.rot, l.heads, n, "latent_q"), B200_OP_LATENT_QUERY, proj, g->pos, cn, g->cells));
                ql->src[4] = ukv;
                ql->src[5] = cache;
                ggml_tensor *part = set(b.op(b.alloc(B200_TYPE_F32, (R + 2) * l.heads, splits, n, "latent_part"), B200_OP_LATENT_DECODE, ql, g->pos, cache, g->row_seg));
                part->src[4] = g->seg;
                part->src[5] = g->tab;
                mixed = set(b.op(b.alloc(b.act, l.heads * l.vdim, n, 1, "latent_out"), B200_OP_LATENT_VALUE, part, g->pos, ukv, proj));
                mixed->src[4] = sink;
            } else {
                set(b.op(b.alias_of(cache), B200_OP_LATENT_STORE, proj, g->pos, cn, g->cells));
                ggml_tensor *rows = b.take_rows(dtype, cache, g->tab, 1.0f, nullptr, "latent_rows");
                ggml_tensor *kv = b.dense(b.alloc(dtype, ukv->ne[1], g->tab->ne[0], 1, "latent_kv"), ukv, b.view_2d(rows, R, g->tab->ne[0], rows->nb[1], 0),
                                          nullptr, nullptr, 0);
                mixed = set(b.op(b.alloc(b.act, l.heads * l.vdim, n, 1, "latent_out"), B200_OP_LATENT_ATTN, proj, g->pos, kv, rows));
                mixed->src[4] = sink;
                mixed->src[5] = g->seg;
            }
        }
        x = b.dense(b.over(next_slot(), "mix_out"), W(p + "mix.o"), mixed, x, nullptr, 0);
        if (l.ff > 0) {
            ggml_tensor *up = b.normed_dense(W(p + "mlp.up"), x, W(p + "norm2"), b.act, 1, "ff_up");
            x = b.dense(b.over(next_slot(), "l_out"), W(p + "mlp.down"), up, x, nullptr, 0);
        }
    }
    b.off = layer_base;
    x = b.get_rows(x, g->out_ids, "result_rows");
    b.few = s.n_out <= FEW_ROWS;
    b.act = dtype == B200_TYPE_F32 || b.few ? B200_TYPE_F32 : B200_TYPE_BF16;
    g->logits = b.normed_dense(W("head"), x, W("final.norm"), B200_TYPE_F32, 0, "result_output");
    g->argmax = b.op(b.alloc(B200_TYPE_I32, s.n_out, 1, 1, "argmax"), GGML_OP_ARGMAX, g->logits);
    g->bytes = b.high;
    return B200_STATUS_SUCCESS;
}

}  // namespace

std::unique_ptr<Arch> rukusun_from_config(const Json &config, int dtype, std::string *err) {
    std::unique_ptr<RukusunArch> a(new RukusunArch());
    Field f{err};
    a->dtype = dtype;
    a->vocab = f.size(config, "vocab", "model");
    a->width = f.size(config, "width", "model");
    if (const Json *norm = f.get(config, "norm", "model")) a->eps = (float)f.number(*norm, "eps", "norm");
    if (const Json *emb = config.find("embedding"))
        if (emb->find("scale")) a->embed_scale = (float)f.number(*emb, "scale", "embedding");
    const Json *layers = f.get(config, "layers", "model");
    if (layers && layers->items.empty() && err->empty()) *err = "config: no layers";
    for (const Json &j : layers ? layers->items : std::vector<Json>()) {
        Layer l;
        const Json *type = f.get(j, "type", "layer"), *mix = f.get(j, "mixer", "layer");
        if (!type || !mix) break;
        l.heads = f.size(*mix, "heads", "mixer");
        l.dim = f.size(*mix, "dim", "mixer");
        l.vdim = f.size(*mix, "vdim", "mixer");
        if (type->str == "gla") {
            l.type = GLA;
            l.tau = (float)f.number(*mix, "tau", "mixer");
            if (!(l.tau > 0.0f) && err->empty()) *err = "config: tau must be positive";
        } else if (type->str == "latent_attention") {
            l.type = LATENT;
            l.kv_rank = f.size(*mix, "kv_rank", "mixer");
            l.rot = f.size(*mix, "rot_dim", "mixer", 0);
            l.scale = (float)f.number(*mix, "scale", "mixer");
            const Json *rot = mix->find("rot");
            l.rot_dims = l.rot;
            if (rot && !rot->is_null()) {
                l.rot_base = (float)f.number(*rot, "base", "rot");
                if (rot->find("dims")) l.rot_dims = f.size(*rot, "dims", "rot", 0);
            } else {
                l.rot_dims = 0;
            }
            if ((l.rot_dims % 2 || l.rot_dims > l.rot) && err->empty()) *err = "config: rotated dimensions must be an even part of rot_dim";
            const Json *mask = mix->find("mask");
            if (mask && !mask->is_null()) l.window = f.size(*mask, "size", "mask");
        } else if (err->empty()) {
            *err = "config: layer type '" + type->str + "' is not known";
        }
        const Json *mlp = j.find("mlp");
        if (mlp && !mlp->is_null()) {
            const Json *kind = mlp->find("kind");
            if ((!kind || kind->str != "dense") && err->empty()) *err = "config: only dense feed-forwards are known";
            l.ff = f.size(*mlp, "ff", "mlp");
        }
        a->layers.push_back(l);
    }
    a->loop = f.loop(config, (int64_t)a->layers.size());
    if (!err->empty()) return nullptr;
    return a;
}

}  // namespace b200
