// What the decode driver (llama_decode.cpp) and the architectures it serves (arch_*.cpp) share: the context, the graph builder
// over the backend plug-in's tensors, and the interface an architecture implements.
#pragma once
#include <algorithm>
#include <cstdio>
#include <cstring>
#include <deque>
#include <map>
#include <memory>
#include <set>
#include <string>
#include <tuple>
#include <vector>

#include "common.cuh"
#include "ggml_b200_backend.h"
#include "json.h"
#include "llama_b200.h"
#include "tp.h"

namespace b200 {

constexpr size_t TENSOR_ALIGN = 256;
constexpr int64_t KV_PAD = 256;   // crates/llama/src/kv_cache.rs:1887-1917: n_kv is padded to 256 cells

inline size_t plain_type_size(int type) {
    switch (type) {
        case B200_TYPE_F32: case B200_TYPE_I32: return 4;
        case B200_TYPE_F16: case B200_TYPE_BF16: return 2;
        case B200_TYPE_I64: return 8;
        default: return 0;
    }
}
inline size_t quant_row_bytes(int type, int64_t ne0) { return (size_t)(ne0 / GROUP_K) * group_src_bytes(type); }

struct Weight {
    ggml_tensor t;
    ggml_backend_buffer_t buf = nullptr;
};

// What a step's graph is built for; equal shapes share one graph
struct StepShape {
    int64_t n = 0;          // tokens
    int64_t n_out = 0;      // rows whose logits are wanted
    int64_t n_kv = 0;       // masked cache: cells the attention spans
    int64_t n_seg = 0;      // sequences in the step
    int64_t n_tab = 0;      // cells listed for them (padded)
    int64_t max_keys = 0;   // most keys one token sees (padded)
    int64_t max_rows = 0;   // 1: one token per sequence; else the most rows a sequence brings, rounded up to a power of two
    bool operator<(const StepShape &o) const {
        return std::tie(n, n_out, n_kv, n_seg, n_tab, max_keys, max_rows) < std::tie(o.n, o.n_out, o.n_kv, o.n_seg, o.n_tab, o.max_keys, o.max_rows);
    }
};

struct Graph {
    std::deque<ggml_tensor> tensors;      // stable addresses
    std::vector<ggml_tensor *> nodes;
    ggml_tensor *tokens = nullptr, *pos = nullptr, *mask = nullptr, *row_idx = nullptr, *out_ids = nullptr;
    ggml_tensor *seg = nullptr, *row_seg = nullptr, *cells = nullptr, *tab = nullptr;
    ggml_tensor *prev = nullptr;          // the token before each token in its sequence, -1 for the first (null: not wanted)
    ggml_tensor *logits = nullptr, *argmax = nullptr;
    size_t bytes = 0;                     // compute-buffer bytes the graph spans
};

// Where a tensor of the model's files goes: rows row0, row0 + row_step, .. of the device tensor `dst` ([ne0, ne1] of `type`)
struct TensorPlace {
    std::string dst;
    int type = 0;
    int64_t ne0 = 0, ne1 = 0, row0 = 0, rows = 0, row_step = 1;
    bool plus_one = false;   // the file holds the distance from one
};

// What an architecture supplies.  One object per context; the driver owns the weights, the cells, the state slots, the step's
// inputs and the compute buffer.
class Arch {
public:
    virtual ~Arch() {}
    virtual const char *name() const = 0;
    virtual int32_t n_vocab() const = 0;
    // true: attention reads the whole unified cache under an F16 mask.  false: the step's sequences are described by segments
    // and lists of cells, a sequence's tokens arrive in order, and recurrent layers keep a state per slot.
    virtual bool masked_cache() const = 0;
    // segmented architectures: how many positions back any layer looks, the token itself included (0: everything; -1: no
    // layer keeps keys).  Cells further back are given back as the sequence grows.
    virtual int64_t key_span() const { return 0; }
    // with a key_span above 0: how many of a sequence's first positions every later token may see all the same.  Their cells stay.
    virtual int64_t kept_first() const { return 0; }
    virtual int alloc_memory(b200_llama *c) = 0;
    virtual int build(b200_llama *c, Graph *g, uint8_t *base, const StepShape &shape) = 0;
    // the shapes the compute buffer has to hold
    virtual std::vector<StepShape> largest(const b200_llama *c) const = 0;
    // false: the model has no tensor of that name
    virtual bool place(const std::string &, TensorPlace *) const { return false; }
    virtual std::vector<std::string> tensor_names() const { return {}; }
    // a tensor is about to be set: what only its shape tells; false when it contradicts what is known
    virtual bool learn_shape(const std::string &, int64_t, int64_t) { return true; }
};
std::unique_ptr<Arch> make_llama_arch(const b200_llama_hparams &hp);
// nullptr and *err when the configuration does not describe a model of the architecture; dtype: B200_TYPE_BF16 / B200_TYPE_F32
typedef std::unique_ptr<Arch> (*ArchFromConfig)(const Json &config, int dtype, std::string *err);
std::unique_ptr<Arch> rukusun_from_config(const Json &config, int dtype, std::string *err);
std::unique_ptr<Arch> lenolix_from_config(const Json &config, int dtype, std::string *err);

// A sequence of a segmented architecture: the cells of the first positions it keeps for good, those of its positions from `kept` on
// (what stands between has been given back), its next position, its last token and its state slot.
struct Sequence {
    std::vector<int32_t> first_cells, cells;
    int64_t kept = 0;
    int64_t next_pos = 0;
    int32_t last_token = -1;
    int32_t slot = -1;
};

}  // namespace b200

struct b200_llama {
    b200_llama_hparams hp;                // llama architecture only
    std::unique_ptr<b200::Arch> arch;
    int32_t n_ctx = 0, n_batch = 0, n_seq = 1;
    ggml_backend_dev_t dev = nullptr;
    ggml_backend_t backend = nullptr;
    ggml_backend_buffer_type_t buft = nullptr;
    void *stream = nullptr;
    std::map<std::string, std::unique_ptr<b200::Weight>> weights;
    std::set<std::string> tensors_set;    // placed tensors set so far (a device tensor may be put together from several)
    ggml_backend_buffer_t kv_buf = nullptr, compute_buf = nullptr;
    std::vector<ggml_tensor> k_l, v_l;    // llama: [n_embd_k_gqa, n_ctx] F16 per layer
    std::vector<ggml_tensor> mem_l;       // segmented architectures: per layer run its cell rows or its state slots
    // The unified cache's cells: the position and sequence each holds, -1 = free.  A token takes the lowest free cell.
    std::vector<int32_t> cell_pos;
    std::vector<int32_t> cell_seq;
    int32_t used = 0;                     // cells in use
    int32_t high = 0;                     // one past the highest cell in use
    int32_t first_free = 0;               // no free cell below this one
    std::map<int32_t, b200::Sequence> seqs;
    std::vector<int32_t> slot_seq;        // the sequence each state slot serves, -1 = free
    std::map<b200::StepShape, std::unique_ptr<b200::Graph>> graphs;
    b200::Graph *last = nullptr;
    std::vector<uint16_t> mask_host;
    std::vector<int64_t> idx_host;
    std::vector<int32_t> seg_host, row_seg_host, cells_host, tab_host, prev_host;
    // tensor parallel: this rank holds n_head / tp_size heads, n_head_kv / tp_size cache heads, the matching
    // rows / columns of every matrix (tp.cpp) and 1 / tp_size of the vocabulary rows
    int32_t tp_rank = 0, tp_size = 1;
    b200::TpGroup *tp = nullptr;
    std::vector<uint8_t> shard_tmp;
};

namespace b200 {

inline void init_tensor(ggml_tensor *t, int type, int64_t ne0, int64_t ne1 = 1, int64_t ne2 = 1, int64_t ne3 = 1) {
    memset(t, 0, sizeof(*t));
    t->type = type;
    t->ne[0] = ne0; t->ne[1] = ne1; t->ne[2] = ne2; t->ne[3] = ne3;
    const size_t row = is_quant_type(type) ? quant_row_bytes(type, ne0) : plain_type_size(type) * (size_t)ne0;
    t->nb[0] = is_quant_type(type) ? (size_t)group_src_bytes(type) / (type == B200_TYPE_Q4_K || type == B200_TYPE_Q6_K ? 1 : 8) : plain_type_size(type);
    t->nb[1] = row;
    t->nb[2] = t->nb[1] * (size_t)ne1;
    t->nb[3] = t->nb[2] * (size_t)ne2;
}

// One pass over the compute buffer: tensors are placed back to back; a layer's intermediates are
// placed again over the previous layer's (everything runs in order on one stream).
struct Builder {
    b200_llama *c;
    Graph *g;
    uint8_t *base;
    size_t off = 0, high = 0;

    ggml_tensor *fresh(int type, int64_t ne0, int64_t ne1 = 1, int64_t ne2 = 1, int64_t ne3 = 1) {
        g->tensors.emplace_back();
        ggml_tensor *t = &g->tensors.back();
        init_tensor(t, type, ne0, ne1, ne2, ne3);
        return t;
    }
    ggml_tensor *alloc(int type, int64_t ne0, int64_t ne1 = 1, int64_t ne2 = 1, const char *name = "") {
        ggml_tensor *t = fresh(type, ne0, ne1, ne2);
        off = (off + TENSOR_ALIGN - 1) / TENSOR_ALIGN * TENSOR_ALIGN;
        t->data = base ? base + off : nullptr;
        t->buffer = c->compute_buf;
        off += t->nb[3];
        high = std::max(high, off);
        snprintf(t->name, sizeof(t->name), "%s", name);
        return t;
    }
    ggml_tensor *op(ggml_tensor *t, int code, ggml_tensor *a, ggml_tensor *b = nullptr, ggml_tensor *c2 = nullptr, ggml_tensor *d = nullptr) {
        t->op = code;
        t->src[0] = a; t->src[1] = b; t->src[2] = c2; t->src[3] = d;
        g->nodes.push_back(t);
        return t;
    }
    // an alias of src's bytes with its own shape and strides (RESHAPE / VIEW / PERMUTE nodes)
    ggml_tensor *alias(int code, ggml_tensor *src, size_t offset, const int64_t ne[4], const size_t nb[4], const char *name = "") {
        ggml_tensor *t = fresh(src->type, 1);
        for (int i = 0; i < 4; i++) { t->ne[i] = ne[i]; t->nb[i] = nb[i]; }
        t->view_src = src->view_src ? src->view_src : src;
        t->view_offs = src->view_offs + offset;
        t->data = src->data ? (uint8_t *)src->data + offset : nullptr;
        t->buffer = src->buffer;
        snprintf(t->name, sizeof(t->name), "%s", name);
        return op(t, code, src);
    }
    ggml_tensor *reshape_3d(ggml_tensor *a, int64_t ne0, int64_t ne1, int64_t ne2) {
        const int64_t ne[4] = {ne0, ne1, ne2, 1};
        const size_t es = a->nb[0];
        const size_t nb[4] = {es, es * ne0, es * ne0 * ne1, es * ne0 * ne1 * ne2};
        return alias(GGML_OP_RESHAPE, a, 0, ne, nb);
    }
    ggml_tensor *reshape_2d(ggml_tensor *a, int64_t ne0, int64_t ne1) { return reshape_3d(a, ne0, ne1, 1); }
    ggml_tensor *view_2d(ggml_tensor *a, int64_t ne0, int64_t ne1, size_t nb1, size_t offset) {
        const int64_t ne[4] = {ne0, ne1, 1, 1};
        const size_t nb[4] = {a->nb[0], nb1, nb1 * ne1, nb1 * ne1};
        return alias(GGML_OP_VIEW, a, offset, ne, nb);
    }
    ggml_tensor *view_3d(ggml_tensor *a, int64_t ne0, int64_t ne1, int64_t ne2, size_t nb1, size_t nb2, size_t offset) {
        const int64_t ne[4] = {ne0, ne1, ne2, 1};
        const size_t nb[4] = {a->nb[0], nb1, nb2, nb2 * ne2};
        return alias(GGML_OP_VIEW, a, offset, ne, nb);
    }
    // permute(a, 0, 2, 1, 3): swap dims 1 and 2
    ggml_tensor *permute_0213(ggml_tensor *a) {
        const int64_t ne[4] = {a->ne[0], a->ne[2], a->ne[1], a->ne[3]};
        const size_t nb[4] = {a->nb[0], a->nb[2], a->nb[1], a->nb[3]};
        return alias(GGML_OP_PERMUTE, a, 0, ne, nb);
    }
    ggml_tensor *mul_mat(ggml_tensor *w, ggml_tensor *x, const char *name = "") {
        return op(alloc(B200_TYPE_F32, w->ne[1], x->ne[1], 1, name), GGML_OP_MUL_MAT, w, x);
    }
    ggml_tensor *binary(int code, ggml_tensor *a, ggml_tensor *b, const char *name = "") {
        return op(alloc(B200_TYPE_F32, a->ne[0], a->ne[1], a->ne[2], name), code, a, b);
    }
    // a new tensor over the bytes of `slot` (the residual stream alternates between two slots)
    ggml_tensor *over(const ggml_tensor *slot, const char *name) {
        ggml_tensor *t = fresh(slot->type, slot->ne[0], slot->ne[1], slot->ne[2]);
        t->data = slot->data;
        t->buffer = slot->buffer;
        snprintf(t->name, sizeof(t->name), "%s", name);
        return t;
    }
    ggml_tensor *rms_norm(ggml_tensor *a, float eps) {
        ggml_tensor *t = op(alloc(B200_TYPE_F32, a->ne[0], a->ne[1], a->ne[2]), GGML_OP_RMS_NORM, a);
        memcpy(&t->op_params[0], &eps, 4);
        return t;
    }
    // crates/llama/src/graph_arch.rs:1119-1122 build_norm_rms
    ggml_tensor *norm(ggml_tensor *a, ggml_tensor *w, float eps, const char *name) { return binary(GGML_OP_MUL, rms_norm(a, eps), w, name); }
    ggml_tensor *silu(ggml_tensor *a) {
        ggml_tensor *t = op(alloc(B200_TYPE_F32, a->ne[0], a->ne[1], a->ne[2]), GGML_OP_UNARY, a);
        t->op_params[0] = GGML_UNARY_OP_SILU;
        return t;
    }
    // crates/ggml/src/ops.rs rope_ext: op_params = [n_past, n_dims, mode, n_ctx, n_ctx_orig, freq_base, freq_scale,
    // ext_factor, attn_factor, beta_fast, beta_slow, sections[4], n_offs]
    ggml_tensor *rope(ggml_tensor *a, ggml_tensor *pos, const char *name) {
        const b200_llama_hparams &hp = c->hp;
        ggml_tensor *t = op(alloc(B200_TYPE_F32, a->ne[0], a->ne[1], a->ne[2], name), GGML_OP_ROPE, a, pos);
        const float f[6] = {hp.rope_freq_base, hp.rope_freq_scale, 0.0f, 1.0f, 32.0f, 1.0f};
        t->op_params[1] = hp.n_embd_head;
        t->op_params[2] = hp.rope_mode;
        t->op_params[4] = hp.n_ctx_train;
        memcpy(&t->op_params[5], f, sizeof(f));
        return t;
    }
    // set_rows(cache, rows, idx): the result aliases the cache tensor
    ggml_tensor *set_rows(ggml_tensor *cache, ggml_tensor *rows, ggml_tensor *idx) {
        ggml_tensor *t = fresh(cache->type, 1);
        for (int i = 0; i < 4; i++) { t->ne[i] = cache->ne[i]; t->nb[i] = cache->nb[i]; }
        t->view_src = cache;
        t->data = cache->data;
        t->buffer = cache->buffer;
        return op(t, GGML_OP_SET_ROWS, rows, idx);
    }
    // the sum of a over the ranks of the tensor-parallel group, in place: the node aliases a
    ggml_tensor *tp_all_reduce(ggml_tensor *a, const char *name) {
        ggml_tensor *t = fresh(a->type, a->ne[0], a->ne[1], a->ne[2]);
        t->data = a->data;
        t->buffer = a->buffer;
        t->view_src = a->view_src ? a->view_src : a;
        t->view_offs = a->view_offs;
        snprintf(t->name, sizeof(t->name), "%s", name);
        return op(t, B200_OP_TP_ALL_REDUCE, a);
    }
    ggml_tensor *get_rows(ggml_tensor *table, ggml_tensor *ids, const char *name = "") {
        return op(alloc(B200_TYPE_F32, table->ne[0], ids->ne[0], 1, name), GGML_OP_GET_ROWS, table, ids);
    }
};

inline ggml_tensor *weight(b200_llama *c, const std::string &name) {
    auto it = c->weights.find(name);
    return it == c->weights.end() ? nullptr : &it->second->t;
}

}  // namespace b200
