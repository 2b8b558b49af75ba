// The llama architecture for the decode driver: one attention / FFN block per layer over the unified F16 cache.
#include <cmath>

#include "decode_ctx.h"

namespace b200 {
namespace {

// crates/llama/src/graph_arch.rs:106-248 with attn_kv_cached's flash-attention branch (:1173-1240) and
// build_ffn_silu_par (:1128-1158).  base == nullptr only measures.
int build_llama(b200_llama *c, Graph *g, uint8_t *base, int64_t n, int64_t n_kv, int64_t n_out) {
    const b200_llama_hparams &hp = c->hp;
    const int64_t E = hp.n_embd, HD = hp.n_embd_head, H = hp.n_head / c->tp_size, HK = hp.n_head_kv / c->tp_size, EK = HK * HD;
    const bool tp = c->tp_size > 1;
    Builder b{c, g, base};
    g->tokens = b.alloc(B200_TYPE_I32, n, 1, 1, "inp_tokens");
    g->pos = b.alloc(B200_TYPE_I32, n, 1, 1, "inp_pos");
    g->mask = b.alloc(B200_TYPE_F16, n_kv, n, 1, "kq_mask");
    g->row_idx = b.alloc(B200_TYPE_I64, n, 1, 1, "kv_idxs");
    g->out_ids = b.alloc(B200_TYPE_I32, n_out, 1, 1, "inp_out_ids");
    ggml_tensor *resid[2] = {b.alloc(B200_TYPE_F32, E, n, 1, "resid_a"), b.alloc(B200_TYPE_F32, E, n, 1, "resid_b")};

    ggml_tensor *tok_embd = weight(c, "token_embd.weight");
    B200_REQUIRE(tok_embd != nullptr, "llama: token_embd.weight has not been set");
    ggml_tensor *inp = b.op(b.over(resid[0], "inp_embd"), GGML_OP_GET_ROWS, tok_embd, g->tokens);
    const size_t layer_base = b.off;
    const float kq_scale = 1.0f / sqrtf((float)HD);

    for (int il = 0; il < hp.n_layer; il++) {
        b.off = layer_base;
        const std::string p = "blk." + std::to_string(il) + ".";
        ggml_tensor *wq = weight(c, p + "attn_q.weight"), *wk = weight(c, p + "attn_k.weight"), *wv = weight(c, p + "attn_v.weight");
        ggml_tensor *wo = weight(c, p + "attn_output.weight"), *an = weight(c, p + "attn_norm.weight"), *fn = weight(c, p + "ffn_norm.weight");
        ggml_tensor *wg = weight(c, p + "ffn_gate.weight"), *wu = weight(c, p + "ffn_up.weight"), *wd = weight(c, p + "ffn_down.weight");
        B200_REQUIRE(wq && wk && wv && wo && an && fn && wg && wu && wd, "llama: layer %d is missing a tensor", il);

        ggml_tensor *cur = b.norm(inp, an, hp.norm_rms_eps, "attn_norm");
        // root 1: the K cache write
        ggml_tensor *k = b.reshape_3d(b.mul_mat(wk, cur, "Kcur"), HD, HK, n);
        k = b.rope(k, g->pos, "Kcur_rope");
        ggml_tensor *k_rows = b.view_2d(k, EK, n, k->nb[2], 0);
        b.set_rows(&c->k_l[il], k_rows, g->row_idx);
        // root 2: the V cache write
        ggml_tensor *v = b.reshape_3d(b.mul_mat(wv, cur, "Vcur"), HD, HK, n);
        ggml_tensor *v_rows = b.view_2d(v, EK, n, v->nb[2], 0);
        b.set_rows(&c->v_l[il], v_rows, g->row_idx);
        // root 3: the layer output, reached through the attention
        ggml_tensor *q = b.reshape_3d(b.mul_mat(wq, cur, "Qcur"), HD, H, n);
        q = b.rope(q, g->pos, "Qcur_rope");
        ggml_tensor *q_fa = b.permute_0213(q);
        // KvCache::get_k / get_v: [head, n_head_kv, n_kv] views of the layer's cache, then [head, n_kv, n_head_kv]
        ggml_tensor *k_fa = b.permute_0213(b.view_3d(&c->k_l[il], HD, HK, n_kv, HD * 2, EK * 2, 0));
        ggml_tensor *v_fa = b.permute_0213(b.view_3d(&c->v_l[il], HD, HK, n_kv, HD * 2, EK * 2, 0));
        ggml_tensor *fa = b.op(b.alloc(B200_TYPE_F32, HD, H, n, "kqv_out"), GGML_OP_FLASH_ATTN_EXT, q_fa, k_fa, v_fa, g->mask);
        memcpy(&fa->op_params[0], &kq_scale, 4);
        ggml_tensor *attn = b.mul_mat(wo, b.reshape_2d(fa, HD * H, n), "attn_out");
        if (tp) attn = b.tp_all_reduce(attn, "attn_out_sum");   // attn holds the partial sums over this rank's heads
        ggml_tensor *ffn_inp = b.binary(GGML_OP_ADD, attn, inp, "ffn_inp");
        cur = b.norm(ffn_inp, fn, hp.norm_rms_eps, "ffn_norm");
        ggml_tensor *gate = b.silu(b.mul_mat(wg, cur, "ffn_gate"));
        ggml_tensor *up = b.mul_mat(wu, cur, "ffn_up");
        ggml_tensor *down = b.mul_mat(wd, b.binary(GGML_OP_MUL, gate, up, "ffn_gate_par"), "ffn_out");
        if (tp) down = b.tp_all_reduce(down, "ffn_out_sum");   // down holds the partial sums over this rank's FFN rows
        inp = b.op(b.over(resid[(il + 1) & 1], "l_out"), GGML_OP_ADD, down, ffn_inp);
    }
    b.off = layer_base;
    ggml_tensor *on = weight(c, "output_norm.weight");
    ggml_tensor *ow = weight(c, "output.weight");
    if (!ow) ow = tok_embd;   // tied embeddings
    B200_REQUIRE(on != nullptr, "llama: output_norm.weight has not been set");
    ggml_tensor *cur = b.norm(inp, on, hp.norm_rms_eps, "result_norm");
    cur = b.get_rows(cur, g->out_ids, "result_norm_rows");   // crates/llama/src/graph.rs:308-313 out_rows
    g->logits = b.mul_mat(ow, cur, "result_output");
    if (tp && ow != tok_embd) {   // this rank's vocabulary rows: gather the full row on every rank
        ggml_tensor *staging = b.alloc(B200_TYPE_F32, ow->ne[1] * c->tp_size, n_out, 1, "result_output_staging");
        g->logits = b.op(b.alloc(B200_TYPE_F32, ow->ne[1] * c->tp_size, n_out, 1, "result_output_all"), B200_OP_TP_ALL_GATHER, g->logits, staging);
    }
    g->argmax = b.op(b.alloc(B200_TYPE_I32, n_out, 1, 1, "argmax"), GGML_OP_ARGMAX, g->logits);
    g->bytes = b.high;
    return B200_STATUS_SUCCESS;
}

class LlamaArch : public Arch {
public:
    explicit LlamaArch(const b200_llama_hparams &hp) : hp_(hp) {}
    const char *name() const override { return "llama"; }
    int32_t n_vocab() const override { return hp_.n_vocab; }
    bool masked_cache() const override { return true; }
    // KV cache: per layer K and V, [n_embd_k_gqa, n_ctx] F16, zero-filled
    int alloc_memory(b200_llama *c) override {
        const int64_t EK = (int64_t)hp_.n_head_kv / c->tp_size * hp_.n_embd_head;
        const size_t per = ((size_t)EK * 2 * c->n_ctx + TENSOR_ALIGN - 1) / TENSOR_ALIGN * TENSOR_ALIGN;
        c->kv_buf = c->buft->iface.alloc_buffer(c->buft, per * 2 * hp_.n_layer);
        if (!c->kv_buf) return B200_STATUS_ALLOC_FAILED;
        c->kv_buf->iface.clear(c->kv_buf, 0);
        c->k_l.resize(hp_.n_layer);
        c->v_l.resize(hp_.n_layer);
        uint8_t *kvb = (uint8_t *)c->kv_buf->iface.get_base(c->kv_buf);
        for (int il = 0; il < hp_.n_layer; il++) {
            for (int which = 0; which < 2; which++) {
                ggml_tensor *t = which ? &c->v_l[il] : &c->k_l[il];
                init_tensor(t, B200_TYPE_F16, EK, c->n_ctx);
                t->buffer = c->kv_buf;
                t->data = kvb + per * (2 * il + which);
                snprintf(t->name, sizeof(t->name), "cache_%c_l%d", which ? 'v' : 'k', il);
            }
        }
        return B200_STATUS_SUCCESS;
    }
    int build(b200_llama *c, Graph *g, uint8_t *base, const StepShape &s) override { return build_llama(c, g, base, s.n, s.n_kv, s.n_out); }
    std::vector<StepShape> largest(const b200_llama *c) const override {
        StepShape s;
        s.n = s.n_out = c->n_batch;
        s.n_kv = c->n_ctx;
        return {s};
    }

private:
    b200_llama_hparams hp_;
};

}  // namespace

std::unique_ptr<Arch> make_llama_arch(const b200_llama_hparams &hp) { return std::unique_ptr<Arch>(new LlamaArch(hp)); }

}  // namespace b200
