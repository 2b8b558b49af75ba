// What the architectures over dense weights (arch_rukusun.cpp, arch_lenolix.cpp) share: the order of layers with a stretch that runs
// several times, nodes of a step, configuration fields.
#pragma once
#include <cmath>

#include "decode_ctx.h"

namespace b200 {

constexpr int64_t FEW_ROWS = 16;   // rows up to which activations stay F32 and mat-muls read the weights row by row

inline int32_t bits(float f) {
    int32_t i;
    memcpy(&i, &f, 4);
    return i;
}

struct LoopSpec {
    int64_t start = 0, stop = 0, times = 0;   // times 0: no loop
};
// the layers in the order they run: (layer, pass); pass -1 outside the loop
inline std::vector<std::pair<int64_t, int64_t>> layer_runs(int64_t n, const LoopSpec &loop) {
    std::vector<std::pair<int64_t, int64_t>> r;
    const int64_t head = loop.times ? loop.start : n;
    for (int64_t i = 0; i < head; i++) r.emplace_back(i, -1);
    for (int64_t t = 0; t < loop.times; t++)
        for (int64_t i = loop.start; i < loop.stop; i++) r.emplace_back(i, t);
    for (int64_t i = loop.times ? loop.stop : n; i < n; i++) r.emplace_back(i, -1);
    return r;
}

// "l<i>.<rest>" of one of n layers
inline bool split_layer_name(const std::string &t, int64_t n, int64_t *il, std::string *pre, std::string *rest) {
    const size_t dot = t.find('.');
    if (t[0] != 'l' || dot == std::string::npos || dot < 2 || dot > 7) return false;
    *il = 0;
    for (size_t i = 1; i < dot; i++) {
        if (t[i] < '0' || t[i] > '9') return false;
        *il = *il * 10 + (t[i] - '0');
    }
    *pre = t.substr(0, dot + 1);
    *rest = t.substr(dot + 1);
    return *il < n;
}

inline int require_tensors(b200_llama *c, const Arch &a) {
    for (const std::string &t : a.tensor_names()) {
        TensorPlace p;
        B200_REQUIRE(c->tensors_set.count(t) && a.place(t, &p) && weight(c, p.dst) != nullptr, "%s: tensor %s has not been set", a.name(), t.c_str());
    }
    return B200_STATUS_SUCCESS;
}

// the nodes of one step
struct StepBuilder : Builder {
    int act;      // type of the rows handed to mat-muls
    bool few;
    float eps;

    ggml_tensor *dense(ggml_tensor *dst, ggml_tensor *w, ggml_tensor *x, ggml_tensor *addend, ggml_tensor *norm_w, int act_code) {
        ggml_tensor *t = op(dst, B200_OP_DENSE_MM, w, x, addend, norm_w);
        t->op_params[0] = act_code;
        t->op_params[1] = bits(eps);
        return t;
    }
    // the inputs the driver fills in
    void inputs(const StepShape &s) {
        g->tokens = alloc(B200_TYPE_I32, s.n, 1, 1, "inp_tokens");
        g->pos = alloc(B200_TYPE_I32, s.n, 1, 1, "inp_pos");
        g->cells = alloc(B200_TYPE_I32, s.n, 1, 1, "inp_cells");
        g->row_seg = alloc(B200_TYPE_I32, s.n, 1, 1, "inp_row_seg");
        g->seg = alloc(B200_TYPE_I32, SEG_FIELDS, s.n_seg, 1, "inp_seg");
        g->tab = alloc(B200_TYPE_I32, std::max<int64_t>(s.n_tab, 1), 1, 1, "inp_tab");
        g->out_ids = alloc(B200_TYPE_I32, s.n_out, 1, 1, "inp_out_ids");
    }
    // w applied to the normed rows: inside the mat-mul while there are few
    ggml_tensor *normed_dense(ggml_tensor *w, ggml_tensor *x, ggml_tensor *norm_w, int type, int act_code, const char *name) {
        if (!few) {
            ggml_tensor *h = op(alloc(act, x->ne[0], x->ne[1]), B200_OP_RMS_NORM_W, x, norm_w);
            h->op_params[0] = bits(eps);
            x = h;
            norm_w = nullptr;
        }
        return dense(alloc(type, w->ne[1], x->ne[1], 1, name), w, x, nullptr, norm_w, act_code);
    }
    ggml_tensor *take_rows(int type, ggml_tensor *table, ggml_tensor *ids, float factor, ggml_tensor *over_slot, const char *name) {
        ggml_tensor *t = op(over_slot ? over(over_slot, name) : alloc(type, table->ne[0], ids->ne[0], 1, name), B200_OP_TAKE_ROWS, table, ids);
        t->op_params[0] = bits(factor);
        return t;
    }
    ggml_tensor *layer_norm(int type, ggml_tensor *x, ggml_tensor *w, ggml_tensor *bias, const char *name) {
        ggml_tensor *t = op(alloc(type, x->ne[0], x->ne[1], 1, name), B200_OP_LAYER_NORM_W, x, w, bias);
        t->op_params[0] = bits(eps);
        return t;
    }
    // the whole of `src` under another node's name (a node that writes into memory it was given)
    ggml_tensor *alias_of(ggml_tensor *src) {
        ggml_tensor *t = fresh(src->type, 1);
        for (int i = 0; i < 4; i++) { t->ne[i] = src->ne[i]; t->nb[i] = src->nb[i]; }
        t->view_src = src;
        t->data = src->data;
        t->buffer = src->buffer;
        return t;
    }
};

// reads a configuration; the first thing that is missing or unusable is kept in *err
struct Field {
    std::string *err;
    const Json *get(const Json &o, const char *key, const char *where) {
        const Json *v = o.find(key);
        if (!v && err->empty()) *err = std::string("config: ") + where + " has no '" + key + "'";
        return v;
    }
    double number(const Json &o, const char *key, const char *where) {
        const Json *v = get(o, key, where);
        if (!v) return 0.0;
        if (v->kind != Json::NUM && err->empty()) *err = std::string("config: ") + where + " '" + key + "' is not a number";
        return v->num;
    }
    int64_t size(const Json &o, const char *key, const char *where, int64_t low = 1) {
        const double v = number(o, key, where);
        if ((v != std::floor(v) || v < (double)low || v > 1e9) && err->empty()) *err = std::string("config: ") + where + " '" + key + "' is not a usable size";
        return (int64_t)v;
    }
    LoopSpec loop(const Json &config, int64_t n_layers) {
        LoopSpec l;
        const Json *j = config.find("loop");
        if (!j || j->is_null()) return l;
        l.start = size(*j, "start", "loop", 0);
        l.stop = size(*j, "stop", "loop");
        l.times = size(*j, "times", "loop");
        if ((l.stop <= l.start || l.stop > n_layers) && err->empty()) *err = "config: the loop's layers are out of range";
        return l;
    }
};

}  // namespace b200
