"""Rukusun on the GPU against the plain decoder (plain_decoder.py, float64): each mechanism alone, prompts against decoding,
portions, batches, cells and slots that are used again, window and chunk edges, other sizes, long decoding, generation through the
serving loop, model folders."""
import importlib
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import b200
import plain_decoder as P
import rukusun_models as M
from decoder_checks import Expected, check, cycle, feed, model, plain_greedy, write_folder

pytestmark = pytest.mark.gpu

@pytest.fixture(scope="module")
def ll():
    b200.load()
    return importlib.import_module("llama_rust_b200.llama")


@pytest.fixture(scope="module")
def engine(ll):
    return importlib.import_module("llama_rust_b200.engine")


STACK = [M.gla(), M.latent(), M.gla(heads=1, dim=32, vdim=8, tau=1.0, ff=0)]


# ---- each mechanism alone, in both forms of a step ----------------------------------------------------------
ALONE = {
    "gla": [M.gla(ff=0)],
    "gla strong decay": [M.gla(tau=0.25, ff=0)],
    "gla slow decay": [M.gla(tau=64.0, ff=0)],
    "latent, window": [M.latent(ff=0)],
    "latent, one key": [M.latent(window=1, ff=0)],
    "latent, no window": [M.latent(window=None, ff=0)],
    "feed-forward": [M.gla(ff=72)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ALONE)
def test_mechanism_alone(ll, name, dtype):
    cfg = M.config(ALONE[name])
    w = M.weights(cfg, 11)
    if name == "feed-forward":
        w["l0.mix.o"] = w["l0.mix.o"] * 0
    toks = M.tokens(cfg, 150, 12)
    want = Expected(cfg, w, toks, dtype)
    m = model(ll, cfg, w, dtype)
    check(feed(m, toks, 150, 0), want, "prompt")
    check(feed(m, toks[:40], 1, 1), want[:40], "decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("loop", [None, (0, 2, 1), (1, 3, 3), (0, 3, 2)])
def test_layer_order_and_loop(ll, loop, dtype):
    cfg = M.config(STACK, loop=loop)
    w, toks = M.weights(cfg, 21), M.tokens(cfg, 90, 22)
    want = Expected(cfg, w, toks, dtype)
    m = model(ll, cfg, w, dtype)
    check(feed(m, toks, cycle(70, 1, 1, 5, 13)), want)


# ---- sizes ---------------------------------------------------------------------------------------------------
SIZES = {
    "odd everywhere": (M.config([M.gla(heads=5, dim=7, vdim=9, ff=33), M.latent(heads=3, dim=5, rot=6, rank=11, vdim=7, window=5, ff=21)], width=37, vocab=53), 3),
    "nothing rotates": (M.config([M.latent(heads=2, dim=16, rot=0, rank=16, vdim=8, window=6)], width=32, vocab=64), 4),
    "one head, one of each": (M.config([M.gla(heads=1, dim=1, vdim=1, ff=1), M.latent(heads=1, dim=1, rot=2, rank=1, vdim=1, window=2, ff=0)], width=16, vocab=31), 1),
    "heads beyond a block's": (M.config([M.latent(heads=19, dim=8, rot=8, rank=16, vdim=8, window=21)], width=64, vocab=77), 4),
    "head 128 x 256": (M.config([M.gla(heads=2, dim=128, vdim=256, tau=16.0), M.latent(heads=2, dim=128, rot=64, rank=512, vdim=128, window=70)], width=96, vocab=203), 16),
    "head 256": (M.config([M.gla(heads=1, dim=256, vdim=64, tau=8.0), M.latent(heads=2, dim=192, rot=64, rank=600, vdim=72, window=40)], width=64, vocab=99), 32),
    "head 300": (M.config([M.gla(heads=1, dim=300, vdim=20, tau=8.0, ff=0), M.latent(heads=1, dim=260, rot=20, rank=36, vdim=140, window=30)], width=64, vocab=99), 70),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", SIZES)
def test_sizes(ll, name, dtype):
    cfg, rank = SIZES[name]
    w, toks = M.weights(cfg, 31, rank=rank, decay=(-1.0, 5.0)), M.tokens(cfg, 100, 32)
    want = Expected(cfg, w, toks, dtype)
    m = model(ll, cfg, w, dtype)
    if name.startswith("one head"):
        want.limit = want.limit * 8   # one number per head: the norms divide by what is left of a single product
    check(feed(m, toks, 100, 0), want, "prompt")
    check(feed(m, toks[:60], cycle(50, 1, 1, 2, 6), 1), want[:60], "portions")


# ---- portions ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2,), (3, 8), (9, 16, 17), (63, 64, 65), (33, 1, 2, 100)])
def test_portions(ll, sizes, dtype):
    cfg = M.config(STACK, loop=(0, 2, 2))
    w, toks = M.weights(cfg, 41), M.tokens(cfg, 203, 42)
    want = Expected(cfg, w, toks, dtype)
    m = model(ll, cfg, w, dtype)
    check(feed(m, toks, cycle(*sizes)), want)


# ---- batches -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_step(ll, dtype):
    cfg = M.config(STACK, loop=(1, 2, 2))
    w = M.weights(cfg, 51)
    lens = [70, 1, 33, 16, 5]
    toks = [M.tokens(cfg, n + 12, 52 + i) for i, n in enumerate(lens)]
    want = [Expected(cfg, w, t, dtype) for t in toks]
    m = model(ll, cfg, w, dtype, n_seq=5)
    at = [0] * 5
    # prompts of every sequence together, then steps that mix single tokens, short and longer portions, some sequences left out
    for step in ([70, 1, 33, 16, 5], [1, 1, 1, 1, 1], [1, 0, 4, 1, 2], [2, 9, 1, 0, 1], [1, 1, 1, 3, 1], [7, 1, 5, 7, 7]):
        rows, pos, seq, spans = [], [], [], []
        for s, n in enumerate(step):
            if n:
                spans.append((s, at[s], n))
            rows += toks[s][at[s]:at[s] + n]
            pos += range(at[s], at[s] + n)
            seq += [s] * n
            at[s] += n
        got, _ = m.decode_seqs(rows, pos, seq, np.arange(len(rows)))
        i = 0
        for s, a, n in spans:
            check(got[i:i + n], want[s][a:a + n], f"sequence {s} at {a}")
            i += n


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_sequences_one_token_each(ll, dtype):
    cfg = M.config(STACK)
    w, n = M.weights(cfg, 61), 24
    toks = [M.tokens(cfg, 14, 62 + i) for i in range(n)]
    want = [Expected(cfg, w, t, dtype) for t in toks]
    m = model(ll, cfg, w, dtype, n_seq=n)
    for t in range(14):
        got, _ = m.decode_seqs([x[t] for x in toks], [t] * n, np.arange(n), np.arange(n))
        for s in range(n):
            check(got[s:s + 1], want[s][t:t + 1], f"sequence {s} at {t}")


# ---- cells and slots used again --------------------------------------------------------------------------------
def test_cells_and_slots_are_used_again(ll):
    cfg = M.config(STACK, loop=(0, 2, 2))
    w = M.weights(cfg, 71)
    m = model(ll, cfg, w, n_ctx=256, n_seq=2)
    a, b, c = (M.tokens(cfg, n, 72 + n) for n in (120, 60, 90))
    pa, pb, pc = (Expected(cfg, w, t) for t in (a, b, c))
    check(feed(m, a[:100], 40, 0), pa[:100])
    used = m.kv_used()
    assert used == 8, "cells out of every window have been given back"   # a window of 9 keeps 8 for the next token
    check(feed(m, b, 7, 1), pb)
    with pytest.raises(b200.load().B200Error):
        feed(m, c[:3], 3, 2)                                # no slot left
    m.seq_rm(1)
    assert m.kv_used() == used
    check(feed(m, c, cycle(64, 3, 1), 2), pc, "in another's slot")
    check(feed(m, a[100:], 1, 0, 100), pa[100:], "the one that stayed")
    m.kv_clear()
    assert m.kv_used() == 0
    check(feed(m, b, 60, 5), pb, "after clearing")
    with pytest.raises(b200.load().B200Error):
        m.decode_seqs([1], [61], [5], [0])                  # not the sequence's next position
    check(feed(m, c[:5], 5, 6), pc[:5], "after a refused step")


def test_a_full_cache_is_refused_and_survives(ll):
    cfg = M.config([M.latent(window=None)])
    w, toks = M.weights(cfg, 75), M.tokens(cfg, 200, 76)
    want = Expected(cfg, w, toks)
    m = model(ll, cfg, w, n_ctx=256, n_batch=256)
    check(feed(m, toks, 200, 0), want)
    with pytest.raises(b200.load().B200Error):
        feed(m, toks[:100], 100, 1)
    m.seq_rm(0)
    check(feed(m, toks, 100, 1), want)


# ---- edges: one key that stands out, just inside and just outside what a token sees ------------------------------
def needle(window):
    """a latent layer and a token whose key all queries want: seen, its value takes over the output"""
    cfg = M.config([M.latent(heads=2, dim=16, rot=4, rank=24, vdim=16, window=window, ff=0)], vocab=60)
    w = M.weights(cfg, 81)
    ch = cfg["width"] - 1
    w["embed"][:, ch] = 0.0
    w["embed"][59] *= 0.25
    w["embed"][59, ch] = 2.0                                # the needle's own channel
    w["l0.mix.dkv"][:, ch] = 0.0
    w["l0.mix.dkv"][0] = 0.0
    w["l0.mix.dkv"][0, ch] = 4.0                            # fills latent 0
    w["l0.mix.uk"][:, 0] = 0.0
    for h in range(2):
        w["l0.mix.uk"][16 * h, 0] = 3.0                     # key channel 0 of both heads
        w["l0.mix.q"][20 * h] = 0.0
    w["l0.mix.q"][[0, 20], 0] = 6.0
    w["embed"][:, 0] = 0.6                                  # every token asks for it
    w["l0.mix.uv"][:, 0] *= 4.0
    return cfg, {k: M.bf16(v) for k, v in w.items()}


@pytest.mark.parametrize("window", [1, 2, 16, 17, 63, 64, 65, 130, 256, 257])
def test_window_edges_in_prompts_and_decoding(ll, window):
    cfg, w = needle(window)
    n = window + 90
    for at in (0, 1, 70):
        toks = M.tokens(cfg, n, 82 + at)
        toks = [t % 59 for t in toks]
        toks[at] = 59
        want = Expected(cfg, w, toks)
        inside, outside = at + window - 1, at + window
        wider = dict(cfg, layers=[dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], mask={"size": window + 1}))])
        off = M.error(P.Plain(wider, w).feed(toks), want.rows)
        assert off[outside] > 0.05, "the needle must show"
        m = model(ll, cfg, w, n_seq=3, n_ctx=1024)
        check(feed(m, toks, n, 0), want, "prompt")
        check(feed(m, toks, cycle(max(1, inside), 1, 1, 1), 1), want, "decoded over the edge")
        check(feed(m, toks, cycle(max(1, inside - 1), 2, 2), 2), want, "short portions over the edge")


def test_window_edges_in_bf16(ll):
    for window in (64, 81):
        cfg, w = needle(window)
        toks = [t % 59 for t in M.tokens(cfg, 200, 85)]
        toks[40] = 59
        want = Expected(cfg, w, toks, "bfloat16")
        m = model(ll, cfg, w, "bfloat16", n_seq=2)
        check(feed(m, toks, 200, 0), want, "prompt")
        check(feed(m, toks, cycle(40 + window - 2, 1, 1, 1, 1, 1), 1), want, "decoded")


def test_far_memory_across_chunks(ll):
    """keys of a slow-decay layer asked for hundreds of tokens later, at and around the recurrence's chunk edges"""
    cfg = M.config([M.gla(heads=2, dim=16, vdim=16, tau=64.0, ff=0)], vocab=60)
    w = M.weights(cfg, 91, decay=(5.0, 8.0))
    w["embed"][59] *= 8.0
    for at in (0, 15, 16, 63, 64, 65, 127):
        toks = [t % 59 for t in M.tokens(cfg, 400, 92 + at)]
        toks[at] = 59
        want = Expected(cfg, w, toks)
        other = P.Plain(cfg, w).feed([t if i != at else 0 for i, t in enumerate(toks)])
        assert M.error(other[-1:], want.rows[-1:]).max() > 1e-3, "the far token must show"
        m = model(ll, cfg, w)
        check(feed(m, toks, cycle(400), 0), want, "prompt")
        check(feed(m, toks, cycle(at + 1, 64, 17, 1), 1), want, "portions")


def test_sink_and_first_tokens(ll):
    """large sinks dominate the first tokens, whose windows are nearly empty"""
    cfg = M.config([M.latent(window=12, ff=0)])
    w, toks = M.weights(cfg, 95), M.tokens(cfg, 20, 96)
    for sinks in (-20.0, 0.0, 6.0, 40.0):
        w["l0.mix.sink"] = np.full(3, sinks, np.float32)
        want = Expected(cfg, w, toks)
        m = model(ll, cfg, w)
        check(feed(m, toks, 20, 0), want, f"sink {sinks}, prompt")
        check(feed(m, toks, 1, 1), want, f"sink {sinks}, decoding")


# ---- long decoding, generation, folders ----------------------------------------------------------------------------
def test_long_decoding(ll):
    cfg = M.config(STACK, loop=(0, 3, 2))
    w, toks = M.weights(cfg, 101), M.tokens(cfg, 420, 102)
    want = Expected(cfg, w, toks)
    m = model(ll, cfg, w, n_ctx=256, n_batch=64, n_seq=1)   # fewer cells than tokens: windows slide over used cells
    check(feed(m, toks, cycle(60, *[1] * 360)), want)


@pytest.mark.parametrize("portion,max_seqs", [(None, 8), (5, 2)])
def test_generation_through_the_serving_loop(ll, engine, portion, max_seqs):
    cfg = M.config(STACK, loop=(1, 3, 2))
    w = M.weights(cfg, 111)
    prompts = [M.tokens(cfg, n, 112 + n) for n in (3, 40, 17, 1, 64)]
    m = model(ll, cfg, w, n_batch=48, n_seq=8)
    got = engine.generate(m, prompts, 12, max_seqs=max_seqs, portion=portion)
    for p, g in zip(prompts, got):
        want, gap = plain_greedy(cfg, w, p, 12)
        assert gap > 1e-4 and g == want
    assert m.kv_used() == 0


def test_programs_over_a_model_folder(tmp_path, ll):
    cfg = M.config(STACK, loop=(0, 2, 2))
    w = M.weights(cfg, 121)
    write_folder(tmp_path, cfg, w)
    env = dict(os.environ, B200_NUMERICS="fast")
    prompts = [M.tokens(cfg, n, 122 + n) for n in (9, 30)]
    out = subprocess.run([sys.executable, os.path.join(b200.ROOT, "bin", "generate"), "--model", str(tmp_path), "--dtype", "float32", "--tokens", "6"] +
                         [x for p in prompts for x in ("--prompt", ",".join(map(str, p)))], capture_output=True, text=True, env=env, timeout=300)
    assert out.returncode == 0, out.stderr
    assert [[int(t) for t in line.split(",")] for line in out.stdout.split()] == [plain_greedy(cfg, w, p, 6)[0] for p in prompts]
    toks = M.tokens(cfg, 50, 123)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:47], "want": [46, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[47:49], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[49:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks[:5], "want": [4]}], "end": ["b"]}]
    for dtype in ("float32", "bfloat16"):
        run = subprocess.run([os.path.join(b200.ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "64"],
                             input="\n".join(map(json.dumps, steps)), capture_output=True, text=True, env=env, timeout=300)
        assert run.returncode == 0, run.stderr
        assert [x for x in run.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        assert not os.path.exists(tmp_path / "1.f32")
        want = Expected(cfg, w, toks, dtype)
        for step, rows in ((0, [46, 3]), (2, [49]), (3, [4])):
            check(np.fromfile(tmp_path / f"{step}.f32", np.float32).reshape(len(rows), -1), want[rows], f"step {step}")


def test_missing_and_misshapen_tensors_are_refused(ll):
    mod = b200.load()
    cfg = M.config([M.gla(), M.latent()])
    w = M.weights(cfg, 131)
    m = ll.Model(cfg, 256, 32, dtype="float32")
    with pytest.raises(mod.B200Error):
        m.set_tensors({"l0.mix.q": w["l0.mix.q"]})          # its matrix's size is not known before the decay's rank is
    with pytest.raises(mod.B200Error):
        m.set_tensors({"l1.mix.o": w["l1.mix.o"][:-1]})
    with pytest.raises(mod.B200Error):
        m.set_tensors({"l7.norm1": w["l0.norm1"]})
    m.set_tensors({k: v for k, v in w.items() if k != "l1.mix.uv"})
    with pytest.raises(mod.B200Error, match="l1.mix.uv"):
        m.decode_seqs([1], [0], [0], [0])
    m.set_tensors({"l1.mix.uv": w["l1.mix.uv"]})
    toks = M.tokens(cfg, 10, 132)
    m.kv_clear()
    check(feed(m, toks, 10), Expected(cfg, w, toks))
