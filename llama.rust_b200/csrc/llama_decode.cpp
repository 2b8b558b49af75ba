// A decode driver over the ggml backend plug-in (include/llama_b200.h).
//
// The reference's DecodeContext (crates/llama/src/context.rs) owns the weights, the KV cache and the
// per-step input tensors, builds the forward graph and hands it to a backend.  This file does the same
// with this library's own backend, and it talks to that backend only
// through the vtables a foreign host would use: get_alloc_size / alloc_buffer / set_tensor /
// graph_compute / get_tensor_async.  The nodes of a step come from the context's architecture (arch_*.cpp).
#include <cmath>

#include "decode_ctx.h"

using namespace b200;

namespace {

int64_t n_kv_for(const b200_llama *c, int32_t high) {
    // min(size, max(256, pad256(highest used cell + 1))): crates/llama/src/kv_cache.rs:1887-1917
    const int64_t padded = (high + KV_PAD - 1) / KV_PAD * KV_PAD;
    return std::min<int64_t>(c->n_ctx, std::max<int64_t>(KV_PAD, padded));
}

void set_input(ggml_tensor *t, const void *data, size_t bytes) { t->buffer->iface.set_tensor(t->buffer, t, data, 0, bytes); }
// the per-step inputs: ordered on the backend's stream ahead of the step's graph, no wait per copy
void set_input_async(ggml_backend_t be, ggml_tensor *t, const void *data, size_t bytes) {
    if (be->iface.set_tensor_async) be->iface.set_tensor_async(be, t, data, 0, bytes);
    else set_input(t, data, bytes);
}

// graph_compute over the first `total` nodes: the whole step is one node list, the collectives of a tensor-parallel
// group are nodes of it (B200_OP_TP_*), so the backend can capture and replay the step as one CUDA graph
int run_graph(b200_llama *c, Graph *g, int total) {
    ggml_cgraph cg;
    memset(&cg, 0, sizeof(cg));
    cg.size = cg.n_nodes = total;
    cg.nodes = g->nodes.data();
    return c->backend->iface.graph_compute(c->backend, &cg);
}

}  // namespace

extern "C" {

int b200_llama_new(const b200_llama_hparams *hp, int device, int32_t n_ctx, int32_t n_batch, int32_t cpu_threads, b200_llama **out) {
    return b200_llama_new_tp(hp, device, n_ctx, n_batch, cpu_threads, 0, 1, nullptr, out);
}

static int llama_new_impl(const b200_llama_hparams *hp, int device, int32_t n_ctx, int32_t n_batch, int32_t cpu_threads, int32_t tp_rank,
                          int32_t tp_size, const void *id128, b200_tp_hook_fn hook, void *hook_user, b200_llama **out);

int b200_llama_new_tp(const b200_llama_hparams *hp, int device, int32_t n_ctx, int32_t n_batch, int32_t cpu_threads, int32_t tp_rank,
                      int32_t tp_size, const void *id128, b200_llama **out) {
    return llama_new_impl(hp, device, n_ctx, n_batch, cpu_threads, tp_rank, tp_size, id128, nullptr, nullptr, out);
}

int b200_llama_new_tp_hook(const b200_llama_hparams *hp, int device, int32_t n_ctx, int32_t n_batch, int32_t cpu_threads, int32_t tp_rank,
                           int32_t tp_size, b200_tp_hook_fn hook, void *user, b200_llama **out) {
    B200_REQUIRE(hook != nullptr && tp_size >= 2, "llama_new_tp_hook: needs a hook and at least two ranks");
    return llama_new_impl(hp, device, n_ctx, n_batch, cpu_threads, tp_rank, tp_size, nullptr, hook, user, out);
}

int b200_llama_tp_exchange_kind(const b200_llama *c) {
    if (!c || !c->tp || c->tp->hook) return -1;
    return c->tp->ll_ready ? 1 : 0;
}

// the context of an architecture: backend, memory, cells and slots
static int context_new(std::unique_ptr<Arch> arch, int device, int32_t n_ctx, int32_t n_batch, int32_t n_seq, int32_t cpu_threads, int32_t tp_rank,
                       int32_t tp_size, const void *id128, b200_tp_hook_fn hook, void *hook_user, const b200_llama_hparams *hp, b200_llama **out) {
    B200_REQUIRE(n_ctx > 0 && n_ctx % KV_PAD == 0, "llama_new: n_ctx %d must be a positive multiple of 256", n_ctx);
    B200_REQUIRE(n_batch > 0 && n_batch <= n_ctx, "llama_new: n_batch %d out of (0, n_ctx]", n_batch);
    B200_REQUIRE(n_seq > 0 && n_seq <= 65536, "llama_new: n_seq %d out of range", n_seq);
    ggml_backend_reg_t reg = ggml_backend_init();
    B200_REQUIRE(reg != nullptr && reg->api_version == GGML_BACKEND_API_VERSION, "llama_new: backend registry unavailable");
    ggml_backend_dev_t dev = reg->iface.get_device(reg, (size_t)device);
    B200_REQUIRE(dev != nullptr, "llama_new: no usable device %d", device);
    std::unique_ptr<b200_llama> c(new b200_llama());
    if (hp) c->hp = *hp;
    else memset(&c->hp, 0, sizeof(c->hp));
    c->arch = std::move(arch);
    c->n_ctx = n_ctx;
    c->n_batch = n_batch;
    c->n_seq = n_seq;
    c->dev = dev;
    c->tp_rank = tp_rank;
    c->tp_size = tp_size;
    const std::string params = "cpu_threads=" + std::to_string(cpu_threads > 0 ? cpu_threads : 8);
    c->backend = dev->iface.init_backend(dev, params.c_str());
    if (!c->backend) return B200_STATUS_BACKEND_ERROR;
    c->buft = dev->iface.get_buffer_type(dev);
    typedef void *(*get_stream_fn)(ggml_backend_t);
    get_stream_fn get_stream = (get_stream_fn)reg->iface.get_proc_address(reg, "b200_backend_get_stream");
    c->stream = get_stream ? get_stream(c->backend) : nullptr;
    int rc = c->arch->alloc_memory(c.get());
    if (rc != B200_STATUS_SUCCESS) { b200_llama_free(c.release()); return rc; }
    c->cell_pos.assign(n_ctx, -1);
    c->cell_seq.assign(n_ctx, -1);
    c->slot_seq.assign(n_seq, -1);
    if (tp_size > 1) {
        rc = tp_group_create(tp_rank, tp_size, device, id128, hook, hook_user, &c->tp);
        if (rc != B200_STATUS_SUCCESS) { b200_llama_free(c.release()); return rc; }
        typedef void (*set_tp_fn)(ggml_backend_t, void *);
        set_tp_fn set_tp = (set_tp_fn)reg->iface.get_proc_address(reg, "b200_backend_set_tp");
        if (!set_tp) { b200_llama_free(c.release()); B200_REQUIRE(false, "llama_new: the backend has no tensor-parallel entry"); }
        set_tp(c->backend, c->tp);
    }
    *out = c.release();
    return B200_STATUS_SUCCESS;
}

static int llama_new_impl(const b200_llama_hparams *hp, int device, int32_t n_ctx, int32_t n_batch, int32_t cpu_threads, int32_t tp_rank,
                          int32_t tp_size, const void *id128, b200_tp_hook_fn hook, void *hook_user, b200_llama **out) {
    B200_REQUIRE(hp != nullptr && out != nullptr, "llama_new: null argument");
    *out = nullptr;
    B200_REQUIRE(tp_size >= 1 && tp_rank >= 0 && tp_rank < tp_size, "llama_new: rank %d of %d", tp_rank, tp_size);
    B200_REQUIRE(tp_size == 1 || id128 != nullptr || hook != nullptr, "llama_new: a tensor-parallel group needs the shared id");
    B200_REQUIRE(hp->n_head % tp_size == 0 && hp->n_head_kv % tp_size == 0, "llama_new: %d / %d heads do not split %d ways", hp->n_head,
                 hp->n_head_kv, tp_size);
    B200_REQUIRE(hp->n_vocab > 0 && hp->n_embd > 0 && hp->n_head > 0 && hp->n_head_kv > 0 && hp->n_layer > 0 && hp->n_ff > 0,
                 "llama_new: non-positive model dimension");
    B200_REQUIRE(hp->n_head % hp->n_head_kv == 0, "llama_new: n_head %d is not a multiple of n_head_kv %d", hp->n_head, hp->n_head_kv);
    B200_REQUIRE(hp->n_embd_head == 64 || hp->n_embd_head == 128, "llama_new: head size %d is not 64 or 128", hp->n_embd_head);
    B200_REQUIRE(hp->n_embd % GROUP_K == 0 && hp->n_ff % GROUP_K == 0 && (hp->n_head * hp->n_embd_head) % GROUP_K == 0,
                 "llama_new: n_embd, n_ff and n_head * head size must be multiples of 256");
    B200_REQUIRE(hp->rope_mode == 0 || hp->rope_mode == 2, "llama_new: rope mode %d is neither NORMAL (0) nor NEOX (2)", hp->rope_mode);
    B200_REQUIRE((hp->n_head / tp_size * hp->n_embd_head) % GROUP_K == 0 && (hp->n_ff / tp_size) % GROUP_K == 0 && hp->n_ff % tp_size == 0,
                 "llama_new: a rank's share of the heads and of n_ff must be multiples of 256 elements");
    return context_new(make_llama_arch(*hp), device, n_ctx, n_batch, n_ctx, cpu_threads, tp_rank, tp_size, id128, hook, hook_user, hp, out);
}

// ---- architectures described by a configuration file -------------------------------------------------------
static const struct { const char *name; ArchFromConfig from_config; } CONFIG_ARCHS[] = {
    {"Rukusun", rukusun_from_config},
    {"Lenolix", lenolix_from_config},
};

int b200_model_new(const char *config_json, int dtype, int device, int32_t n_ctx, int32_t n_batch, int32_t n_seq, b200_llama **out) {
    B200_REQUIRE(config_json != nullptr && out != nullptr, "model_new: null argument");
    *out = nullptr;
    B200_REQUIRE(dtype == B200_TYPE_BF16 || dtype == B200_TYPE_F32, "model_new: weights are kept in BF16 or F32, not type %d", dtype);
    Json config;
    B200_REQUIRE(Json::parse(config_json, strlen(config_json), &config) && config.kind == Json::OBJ, "model_new: the configuration is not a JSON object");
    const Json *name = config.find("architecture");
    B200_REQUIRE(name != nullptr && name->kind == Json::STR, "model_new: the configuration names no architecture");
    for (const auto &e : CONFIG_ARCHS) {
        if (name->str != e.name) continue;
        std::string err;
        std::unique_ptr<Arch> arch = e.from_config(config, dtype, &err);
        B200_REQUIRE(arch != nullptr, "model_new: %s", err.c_str());
        // a context's memory depends on the sizes in the configuration alone
        return context_new(std::move(arch), device, n_ctx, n_batch, n_seq, 0, 0, 1, nullptr, nullptr, nullptr, nullptr, out);
    }
    B200_REQUIRE(false, "model_new: architecture %s is not one of this library's", name->str.c_str());
}

int32_t b200_llama_n_vocab(const b200_llama *c) { return c ? c->arch->n_vocab() : 0; }
const char *b200_llama_arch_name(const b200_llama *c) { return c ? c->arch->name() : ""; }
int32_t b200_llama_n_tensors(const b200_llama *c) { return c ? (int32_t)c->arch->tensor_names().size() : 0; }
int b200_llama_learn_shape(b200_llama *c, const char *name, int64_t ne0, int64_t ne1) {
    B200_REQUIRE(c != nullptr && name != nullptr, "llama_learn_shape: null argument");
    B200_REQUIRE(c->arch->learn_shape(name, ne0, ne1), "llama_learn_shape: %s [%lld, %lld] contradicts an earlier tensor", name, (long long)ne1, (long long)ne0);
    return B200_STATUS_SUCCESS;
}

void b200_llama_free(b200_llama *c) {
    if (!c) return;
    if (c->backend) c->backend->iface.synchronize(c->backend);
    c->graphs.clear();
    if (c->compute_buf) c->compute_buf->iface.free_buffer(c->compute_buf);
    if (c->kv_buf) c->kv_buf->iface.free_buffer(c->kv_buf);
    for (auto &kv : c->weights)
        if (kv.second->buf) kv.second->buf->iface.free_buffer(kv.second->buf);
    if (c->backend) c->backend->iface.free(c->backend);
    if (c->tp) tp_group_destroy(c->tp);
    delete c;
}

static int set_tensor_impl(b200_llama *c, const char *name, int type, int64_t ne0, int64_t ne1, const void *data, size_t nbytes, bool whole);

int b200_llama_set_tensor(b200_llama *c, const char *name, int type, int64_t ne0, int64_t ne1, const void *data, size_t nbytes) {
    return set_tensor_impl(c, name, type, ne0, ne1, data, nbytes, true);
}
int b200_llama_set_tensor_shard(b200_llama *c, const char *name, int type, int64_t ne0, int64_t ne1, const void *data, size_t nbytes) {
    return set_tensor_impl(c, name, type, ne0, ne1, data, nbytes, false);
}

static float host_f32(int type, const void *data, size_t i) {
    if (type == B200_TYPE_F32) return ((const float *)data)[i];
    const uint32_t u = (uint32_t)((const uint16_t *)data)[i] << 16;
    float f;
    memcpy(&f, &u, 4);
    return f;
}
static uint16_t host_bf16(float f) {   // round to nearest, ties to even
    uint32_t u;
    memcpy(&u, &f, 4);
    if ((u & 0x7fffffffu) > 0x7f800000u) return (uint16_t)(u >> 16 | 0x40);
    return (uint16_t)((u + 0x7fffu + (u >> 16 & 1)) >> 16);
}

// A tensor of an architecture that says where its tensors go: converted to the type the device tensor holds and copied to its rows
// there (a device tensor may be put together from several of the model's).
static int set_placed_tensor(b200_llama *c, const char *name, int type, int64_t ne0, int64_t ne1, const void *data, size_t nbytes) {
    B200_REQUIRE(type == B200_TYPE_F32 || type == B200_TYPE_BF16, "llama_set_tensor: %s: type %d is not F32 or BF16", name, type);
    B200_REQUIRE(nbytes == plain_type_size(type) * (size_t)ne0 * (size_t)ne1, "llama_set_tensor: %s: %zu bytes do not hold %lld x %lld elements", name,
                 nbytes, (long long)ne1, (long long)ne0);
    int rc = b200_llama_learn_shape(c, name, ne0, ne1);
    if (rc != B200_STATUS_SUCCESS) return rc;
    TensorPlace p;
    B200_REQUIRE(c->arch->place(name, &p), "llama_set_tensor: %s has no tensor %s", c->arch->name(), name);
    B200_REQUIRE(p.ne1 > 0, "llama_set_tensor: %s is part of a matrix whose size another tensor tells; set that one first", name);
    B200_REQUIRE(ne0 == p.ne0 && ne1 == p.rows, "llama_set_tensor: %s is [%lld, %lld], the configuration asks for [%lld, %lld]", name, (long long)ne1,
                 (long long)ne0, (long long)p.rows, (long long)p.ne0);
    auto it = c->weights.find(p.dst);
    if (it == c->weights.end()) {
        std::unique_ptr<Weight> w(new Weight());
        init_tensor(&w->t, p.type, p.ne0, p.ne1);
        snprintf(w->t.name, sizeof(w->t.name), "%s", p.dst.c_str());
        w->buf = c->buft->iface.alloc_buffer(c->buft, w->t.nb[2] + TENSOR_ALIGN);
        if (!w->buf) return B200_STATUS_ALLOC_FAILED;
        w->buf->usage = GGML_BACKEND_BUFFER_USAGE_WEIGHTS;
        w->t.buffer = w->buf;
        w->t.data = w->buf->iface.get_base(w->buf);
        it = c->weights.emplace(p.dst, std::move(w)).first;
    }
    ggml_tensor *t = &it->second->t;
    const size_t count = (size_t)ne0 * (size_t)ne1, offset = (size_t)p.row0 * t->nb[1];
    std::vector<float> f;
    std::vector<uint16_t> h;
    const void *src = data;
    if (p.type == B200_TYPE_F32 && (type != B200_TYPE_F32 || p.plus_one)) {
        f.resize(count);
        for (size_t i = 0; i < count; i++) f[i] = host_f32(type, data, i) + (p.plus_one ? 1.0f : 0.0f);
        src = f.data();
    } else if (p.type == B200_TYPE_BF16 && type != B200_TYPE_BF16) {
        h.resize(count);
        for (size_t i = 0; i < count; i++) h[i] = host_bf16(((const float *)data)[i]);
        src = h.data();
    }
    c->backend->iface.synchronize(c->backend);
    if (p.row_step == 1) {
        t->buffer->iface.set_tensor(t->buffer, t, src, offset, count * plain_type_size(p.type));
    } else {   // between rows of other tensors: what is there comes to the host and goes back
        const size_t row = t->nb[1], span = row * (size_t)((p.rows - 1) * p.row_step + 1);
        c->shard_tmp.resize(span);
        t->buffer->iface.get_tensor(t->buffer, t, c->shard_tmp.data(), offset, span);
        for (int64_t r = 0; r < p.rows; r++) memcpy(&c->shard_tmp[row * (size_t)(r * p.row_step)], (const uint8_t *)src + row * (size_t)r, row);
        t->buffer->iface.set_tensor(t->buffer, t, c->shard_tmp.data(), offset, span);
    }
    c->tensors_set.insert(name);
    c->graphs.clear();
    c->last = nullptr;
    return B200_STATUS_SUCCESS;
}

static int set_tensor_impl(b200_llama *c, const char *name, int type, int64_t ne0, int64_t ne1, const void *data, size_t nbytes, bool whole) {
    B200_REQUIRE(c != nullptr && name != nullptr && data != nullptr, "llama_set_tensor: null argument");
    B200_REQUIRE(ne0 > 0 && ne1 > 0, "llama_set_tensor: %s has an empty shape", name);
    if (!c->arch->masked_cache()) return set_placed_tensor(c, name, type, ne0, ne1, data, nbytes);
    const bool quant = is_quant_type(type);
    B200_REQUIRE(quant || type == B200_TYPE_F32 || type == B200_TYPE_F16, "llama_set_tensor: %s: type %d is not supported", name, type);
    B200_REQUIRE(!quant || ne0 % GROUP_K == 0, "llama_set_tensor: %s: row length %lld is not a multiple of 256", name, (long long)ne0);
    std::unique_ptr<Weight> w(new Weight());
    init_tensor(&w->t, type, ne0, ne1);
    B200_REQUIRE(nbytes == w->t.nb[2], "llama_set_tensor: %s: %zu bytes given, %zu expected", name, nbytes, w->t.nb[2]);
    if (c->tp_size > 1 && whole) {   // keep this rank's shard of the whole tensor
        int32_t split = 0;
        int64_t l0 = 0, l1 = 0;
        int rc = b200_tp_shard_shape(name, type, ne0, ne1, c->tp_size, &split, &l0, &l1);
        if (rc != B200_STATUS_SUCCESS) return rc;
        if (split != 0) {
            init_tensor(&w->t, type, l0, l1);
            c->shard_tmp.resize(w->t.nb[2]);
            rc = b200_tp_shard_tensor(name, type, ne0, ne1, data, c->tp_rank, c->tp_size, c->shard_tmp.data(), c->shard_tmp.size());
            if (rc != B200_STATUS_SUCCESS) return rc;
            data = c->shard_tmp.data();
            nbytes = c->shard_tmp.size();
        }
    }
    snprintf(w->t.name, sizeof(w->t.name), "%s", name);
    w->buf = c->buft->iface.alloc_buffer(c->buft, c->buft->iface.get_alloc_size(c->buft, &w->t));
    if (!w->buf) return B200_STATUS_ALLOC_FAILED;
    w->buf->usage = GGML_BACKEND_BUFFER_USAGE_WEIGHTS;
    w->t.buffer = w->buf;
    w->t.data = w->buf->iface.get_base(w->buf);
    w->buf->iface.init_tensor(w->buf, &w->t);
    w->buf->iface.set_tensor(w->buf, &w->t, data, 0, nbytes);
    auto old = c->weights.find(name);
    if (old != c->weights.end()) {
        c->backend->iface.synchronize(c->backend);
        old->second->buf->iface.free_buffer(old->second->buf);
    }
    c->weights[name] = std::move(w);
    c->graphs.clear();   // graphs hold pointers to the weight tensors
    c->last = nullptr;
    return B200_STATUS_SUCCESS;
}

int b200_llama_kv_clear(b200_llama *c) {
    B200_REQUIRE(c != nullptr, "llama_kv_clear: null context");
    c->backend->iface.synchronize(c->backend);
    c->kv_buf->iface.clear(c->kv_buf, 0);
    std::fill(c->cell_pos.begin(), c->cell_pos.end(), -1);
    std::fill(c->cell_seq.begin(), c->cell_seq.end(), -1);
    std::fill(c->slot_seq.begin(), c->slot_seq.end(), -1);
    c->seqs.clear();
    c->used = c->high = c->first_free = 0;
    return B200_STATUS_SUCCESS;
}

static void free_cell(b200_llama *c, int32_t cell) {
    c->cell_pos[cell] = c->cell_seq[cell] = -1;
    c->used--;
    c->first_free = std::min(c->first_free, cell);
    while (c->high > 0 && c->cell_seq[c->high - 1] < 0) c->high--;
}

int b200_llama_seq_rm(b200_llama *c, int32_t seq) {
    B200_REQUIRE(c != nullptr && seq >= 0, "llama_seq_rm: bad argument");
    for (int32_t j = c->high - 1; j >= 0; j--)
        if (c->cell_seq[j] == seq) free_cell(c, j);
    auto it = c->seqs.find(seq);
    if (it != c->seqs.end()) {
        if (it->second.slot >= 0) c->slot_seq[it->second.slot] = -1;
        c->seqs.erase(it);
    }
    return B200_STATUS_SUCCESS;
}

int32_t b200_llama_kv_used(const b200_llama *c) { return c ? c->used : 0; }

int b200_llama_get_hparams(const b200_llama *c, b200_llama_hparams *out) {
    B200_REQUIRE(c != nullptr && out != nullptr, "llama_get_hparams: null argument");
    B200_REQUIRE(c->arch->masked_cache(), "llama_get_hparams: %s is described by its configuration", c->arch->name());
    *out = c->hp;
    return B200_STATUS_SUCCESS;
}

int b200_llama_decode(b200_llama *c, const int32_t *tokens, const int32_t *pos, int32_t n, float *logits, int32_t *argmax) {
    B200_REQUIRE(n > 0, "llama_decode: batch size %d out of (0, %d]", n, c ? c->n_batch : 0);
    const int32_t last = n - 1;
    return b200_llama_decode_seqs(c, tokens, pos, nullptr, n, &last, 1, logits, argmax);
}

// A step of a segmented architecture, on the host: the sequences among its rows, checked (a sequence's rows stand together and
// continue it), then their cells and slots, and the inputs the nodes read.  Nothing changes before every check has passed.
static int plan_segments(b200_llama *c, const int32_t *tokens, const int32_t *pos, const int32_t *seq_ids, int32_t n, StepShape *s) {
    struct Seg { int32_t seq, row0, rows; int64_t pos0; };
    std::vector<Seg> segs;
    for (int32_t i = 0; i < n; i++) {
        const int32_t q = seq_ids ? seq_ids[i] : 0;
        B200_REQUIRE(q >= 0, "llama_decode: sequence id %d", q);
        if (!segs.empty() && segs.back().seq == q) {
            B200_REQUIRE(pos[i] == pos[i - 1] + 1, "llama_decode: position %d of sequence %d follows %d", pos[i], q, pos[i - 1]);
            segs.back().rows++;
            continue;
        }
        for (const Seg &o : segs) B200_REQUIRE(o.seq != q, "llama_decode: the rows of sequence %d do not stand together", q);
        const auto it = c->seqs.find(q);
        const int64_t want = it == c->seqs.end() ? 0 : it->second.next_pos;
        B200_REQUIRE(pos[i] == want, "llama_decode: sequence %d continues at position %lld, not %d", q, (long long)want, pos[i]);
        segs.push_back({q, i, 1, pos[i]});
    }
    const int64_t span = c->arch->key_span(), keep = span > 0 ? c->arch->kept_first() : 0;
    int64_t fresh = 0, free_slots = 0;
    for (const Seg &g : segs) fresh += c->seqs.find(g.seq) == c->seqs.end();
    for (int32_t q : c->slot_seq) free_slots += q < 0;
    B200_REQUIRE(fresh <= free_slots, "llama_decode: %lld new sequences, %lld of %d state slots free", (long long)fresh, (long long)free_slots, c->n_seq);
    B200_REQUIRE(span < 0 || c->used + n <= c->n_ctx, "llama_decode: kv cache full (%d used + %d > %d)", c->used, n, c->n_ctx);

    c->seg_host.assign(segs.size() * SEG_FIELDS, 0);
    c->row_seg_host.assign(n, 0);
    c->cells_host.assign(n, 0);
    c->prev_host.assign(n, -1);
    c->tab_host.clear();
    int64_t max_keys = 1, max_rows = 1;
    for (size_t k = 0; k < segs.size(); k++) {
        const Seg &g = segs[k];
        Sequence &q = c->seqs[g.seq];
        const bool is_new = q.slot < 0;
        if (is_new) {
            q.slot = (int32_t)(std::find(c->slot_seq.begin(), c->slot_seq.end(), -1) - c->slot_seq.begin());
            c->slot_seq[q.slot] = g.seq;
            q.kept = keep;
        }
        int32_t *f = &c->seg_host[k * SEG_FIELDS];
        f[SEG_ROW0] = g.row0;
        f[SEG_ROWS] = g.rows;
        f[SEG_SLOT] = q.slot;
        f[SEG_FRESH] = is_new;
        f[SEG_POS0] = (int32_t)g.pos0;
        for (int32_t i = 0; i < g.rows; i++) {
            c->row_seg_host[g.row0 + i] = (int32_t)k;
            c->prev_host[g.row0 + i] = q.last_token;
            q.last_token = tokens[g.row0 + i];
            if (span < 0) continue;
            int32_t cell = c->first_free;
            while (c->cell_seq[cell] >= 0) cell++;
            c->first_free = cell + 1;
            c->cell_pos[cell] = (int32_t)(g.pos0 + i);
            c->cell_seq[cell] = g.seq;
            c->used++;
            c->high = std::max(c->high, cell + 1);
            c->cells_host[g.row0 + i] = cell;
            (g.pos0 + i < keep ? q.first_cells : q.cells).push_back(cell);
        }
        q.next_pos = g.pos0 + g.rows;
        max_rows = std::max<int64_t>(max_rows, g.rows);
        if (span >= 0) {
            // the positions the first row can see, up to the last row's own, behind the ones that are kept for good
            const int64_t key0 = span > 0 ? std::max<int64_t>(keep, g.pos0 - span + 1) : 0, at = (int64_t)c->tab_host.size();
            f[SEG_TAB0] = (int32_t)at;
            f[SEG_KEY0] = (int32_t)key0;
            f[SEG_KEPT] = (int32_t)q.first_cells.size();
            c->tab_host.insert(c->tab_host.end(), q.first_cells.begin(), q.first_cells.end());
            for (int64_t p = key0; p < q.next_pos; p++) c->tab_host.push_back(q.cells[p - q.kept]);
            max_keys = std::max(max_keys, (int64_t)c->tab_host.size() - at);
        }
    }
    s->n_seg = (int64_t)segs.size();
    s->max_rows = 1;
    while (s->max_rows < max_rows) s->max_rows *= 2;
    if (span >= 0) {
        s->n_tab = std::min<int64_t>(((int64_t)c->tab_host.size() + KV_PAD - 1) / KV_PAD * KV_PAD, (c->n_ctx + KV_PAD - 1) / KV_PAD * KV_PAD);
        if (max_rows == 1 && span > 0) max_keys = std::min(max_keys, span + keep);
        s->max_keys = std::min<int64_t>((max_keys + KV_PAD - 1) / KV_PAD * KV_PAD, s->n_tab);
        c->tab_host.resize(s->n_tab, 0);
    }
    return B200_STATUS_SUCCESS;
}
// After a step: cells no later token of the sequence can see are free again.
static void trim_sequences(b200_llama *c, const int32_t *seq_ids, int32_t n) {
    const int64_t span = c->arch->key_span();
    if (span <= 0) return;
    for (int32_t i = 0; i < n; i++) {
        if (i > 0 && (!seq_ids || seq_ids[i] == seq_ids[i - 1])) continue;
        Sequence &q = c->seqs[seq_ids ? seq_ids[i] : 0];
        const int64_t first = std::max<int64_t>(q.kept, q.next_pos - span + 1);
        for (int64_t p = q.kept; p < first; p++) free_cell(c, q.cells[p - q.kept]);
        q.cells.erase(q.cells.begin(), q.cells.begin() + (first - q.kept));
        q.kept = first;
    }
}

int b200_llama_decode_seqs(b200_llama *c, const int32_t *tokens, const int32_t *pos, const int32_t *seq_ids, int32_t n,
                           const int32_t *out_rows, int32_t n_out, float *logits, int32_t *argmax) {
    B200_REQUIRE(c != nullptr && tokens != nullptr && pos != nullptr && out_rows != nullptr, "llama_decode: null argument");
    B200_REQUIRE(n > 0 && n <= c->n_batch, "llama_decode: batch size %d out of (0, %d]", n, c->n_batch);
    B200_REQUIRE(n_out > 0 && n_out <= n, "llama_decode: %d output rows for %d tokens", n_out, n);
    for (int i = 0; i < n; i++)
        B200_REQUIRE(tokens[i] >= 0 && tokens[i] < c->arch->n_vocab(), "llama_decode: token %d out of range", tokens[i]);
    for (int i = 0; i < n_out; i++) B200_REQUIRE(out_rows[i] >= 0 && out_rows[i] < n, "llama_decode: output row %d out of range", out_rows[i]);
    const bool masked = c->arch->masked_cache();

    StepShape shape;
    shape.n = n;
    shape.n_out = n_out;
    if (masked) {
        B200_REQUIRE(c->used + n <= c->n_ctx, "llama_decode: kv cache full (%d used + %d > %d)", c->used, n, c->n_ctx);
        // find_slot + assign: the lowest free cells, in order; a cell remembers its sequence and position
        c->idx_host.resize(n);
        int32_t cell = c->first_free, high = c->high;
        for (int i = 0; i < n; i++, cell++) {
            while (c->cell_seq[cell] >= 0) cell++;
            c->idx_host[i] = cell;
            high = std::max(high, cell + 1);
        }
        shape.n_kv = n_kv_for(c, high);
    } else {
        int rc = plan_segments(c, tokens, pos, seq_ids, n, &shape);
        if (rc != B200_STATUS_SUCCESS) return rc;
    }

    // the graph for this shape, sized and built once
    auto it = c->graphs.find(shape);
    if (it == c->graphs.end()) {
        if (!c->compute_buf) {
            size_t bytes = 0;
            for (const StepShape &s : c->arch->largest(c)) {
                Graph measure;
                int rc = c->arch->build(c, &measure, nullptr, s);
                if (rc != B200_STATUS_SUCCESS) return rc;
                bytes = std::max(bytes, measure.bytes);
            }
            c->compute_buf = c->buft->iface.alloc_buffer(c->buft, bytes + TENSOR_ALIGN);
            if (!c->compute_buf) return B200_STATUS_ALLOC_FAILED;
            c->compute_buf->usage = GGML_BACKEND_BUFFER_USAGE_COMPUTE;
        }
        std::unique_ptr<Graph> g(new Graph());
        int rc = c->arch->build(c, g.get(), (uint8_t *)c->compute_buf->iface.get_base(c->compute_buf), shape);
        if (rc != B200_STATUS_SUCCESS) return rc;
        B200_REQUIRE(g->bytes <= c->compute_buf->size, "llama_decode: graph needs %zu bytes, compute buffer has %zu", g->bytes, c->compute_buf->size);
        it = c->graphs.emplace(shape, std::move(g)).first;
    }
    Graph *g = it->second.get();

    if (masked) {
        for (int i = 0; i < n; i++) {
            const int32_t cell = (int32_t)c->idx_host[i];
            c->cell_pos[cell] = pos[i];
            c->cell_seq[cell] = seq_ids ? seq_ids[i] : 0;
            c->high = std::max(c->high, cell + 1);
        }
        c->used += n;
        c->first_free = (int32_t)c->idx_host[n - 1] + 1;
        // crates/llama/src/graph.rs:704-724 fill_kq_mask_f16 with the sequence test of llama-kv-cache's set_input_kq_mask:
        // 0 where the cell belongs to the query's sequence and holds a position <= the query's, -inf elsewhere
        const int64_t n_kv = shape.n_kv;
        c->mask_host.assign((size_t)n * n_kv, 0xFC00);
        for (int i = 0; i < n; i++) {
            const int32_t s = seq_ids ? seq_ids[i] : 0;
            for (int64_t j = 0; j < c->high; j++)
                if (c->cell_seq[j] == s && c->cell_pos[j] >= 0 && c->cell_pos[j] <= pos[i]) c->mask_host[(size_t)i * n_kv + j] = 0;
        }
    }

    // inputs land with synchronous copies after the previous step has drained
    c->backend->iface.synchronize(c->backend);
    set_input_async(c->backend, g->tokens, tokens, (size_t)n * 4);
    set_input_async(c->backend, g->pos, pos, (size_t)n * 4);
    if (g->prev) set_input_async(c->backend, g->prev, c->prev_host.data(), (size_t)n * 4);
    if (masked) {
        set_input_async(c->backend, g->mask, c->mask_host.data(), c->mask_host.size() * 2);
        set_input_async(c->backend, g->row_idx, c->idx_host.data(), (size_t)n * 8);
    } else {
        set_input_async(c->backend, g->cells, c->cells_host.data(), (size_t)n * 4);
        set_input_async(c->backend, g->row_seg, c->row_seg_host.data(), (size_t)n * 4);
        set_input_async(c->backend, g->seg, c->seg_host.data(), c->seg_host.size() * 4);
        if (!c->tab_host.empty()) set_input_async(c->backend, g->tab, c->tab_host.data(), c->tab_host.size() * 4);
    }
    set_input_async(c->backend, g->out_ids, out_rows, (size_t)n_out * 4);

    int rc = run_graph(c, g, (int)g->nodes.size() - (argmax ? 0 : 1));   // the ARGMAX node is last
    if (rc != B200_STATUS_SUCCESS) return rc;
    c->last = g;
    if (!masked) trim_sequences(c, seq_ids, n);
    if (logits) c->backend->iface.get_tensor_async(c->backend, g->logits, logits, 0, (size_t)c->arch->n_vocab() * n_out * 4);
    if (argmax) c->backend->iface.get_tensor_async(c->backend, g->argmax, argmax, 0, (size_t)n_out * 4);
    c->backend->iface.synchronize(c->backend);
    int code = 0;
    rc = b200_kernel_error(&code);
    if (rc != B200_STATUS_SUCCESS) return rc;
    B200_REQUIRE(code == 0, "llama_decode: a kernel reported error code %d", code);
    return B200_STATUS_SUCCESS;
}

int b200_llama_read_node(b200_llama *c, const char *name, void *out, size_t nbytes) {
    B200_REQUIRE(c != nullptr && name != nullptr && out != nullptr, "llama_read_node: null argument");
    B200_REQUIRE(c->last != nullptr, "llama_read_node: no decode call yet");
    const ggml_tensor *found = nullptr;
    for (const ggml_tensor &t : c->last->tensors)
        if (strcmp(t.name, name) == 0) found = &t;
    B200_REQUIRE(found != nullptr, "llama_read_node: no tensor named %s", name);
    B200_REQUIRE(nbytes <= found->nb[3], "llama_read_node: %s holds %zu bytes, %zu asked", name, found->nb[3], nbytes);
    c->backend->iface.get_tensor_async(c->backend, found, out, 0, nbytes);
    c->backend->iface.synchronize(c->backend);
    return B200_STATUS_SUCCESS;
}

int b200_llama_replay(b200_llama *c, int32_t reps, float *ms) {
    B200_REQUIRE(c != nullptr && ms != nullptr && reps > 0, "llama_replay: bad argument");
    B200_REQUIRE(c->last != nullptr, "llama_replay: no decode call to replay");
    Graph *g = c->last;
    void *e0 = nullptr, *e1 = nullptr;
    int rc = b200_event_create(&e0);
    if (rc == B200_STATUS_SUCCESS) rc = b200_event_create(&e1);
    if (rc == B200_STATUS_SUCCESS) rc = b200_event_record(e0, c->stream);
    for (int i = 0; i < reps && rc == B200_STATUS_SUCCESS; i++) rc = run_graph(c, g, (int)g->nodes.size() - 1);
    if (rc == B200_STATUS_SUCCESS) rc = b200_event_record(e1, c->stream);
    if (rc == B200_STATUS_SUCCESS) rc = b200_event_synchronize(e1);
    if (rc == B200_STATUS_SUCCESS) rc = b200_event_elapsed_ms(e0, e1, ms);
    if (e0) b200_event_destroy(e0);
    if (e1) b200_event_destroy(e1);
    return rc;
}

}  // extern "C"
