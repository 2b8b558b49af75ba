"""Lenolix on the GPU against its plain restatement (plain_lenolix.py, float64): each mechanism alone, prompts against decoding,
portions, batches, cells and slots that are used again, window edges and kept first tokens, other sizes, long decoding, generation through
the serving loop, model folders."""
import importlib
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import b200
import lenolix_models as M
from decoder_checks import Expected, check, cycle, feed, model, plain, plain_greedy, write_folder

pytestmark = pytest.mark.gpu

BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


@pytest.fixture(scope="module")
def ll():
    b200.load()
    return importlib.import_module("llama_rust_b200.llama")


@pytest.fixture(scope="module")
def engine(ll):
    return importlib.import_module("llama_rust_b200.engine")


STACK = [M.layer(), M.layer(heads=3, kv_heads=3, dim=16, vdim=24, window=14, keep=0, rot=16, scaling=None, ff=0), M.layer(heads=6, kv_heads=1, dim=12, vdim=8, window=5, keep=7, rot=4)]


# ---- each mechanism alone, in both forms of a step ----------------------------------------------------------
ALONE = {
    "attention, window and kept tokens": ([M.layer(ff=0)], {}),
    "window without kept tokens": ([M.layer(keep=0, ff=0)], {}),
    "no mask": ([M.layer(window=None, ff=0)], {}),
    "one key and the first": ([M.layer(window=1, keep=1, ff=0)], {}),
    "more kept than the window": ([M.layer(window=4, keep=30, ff=0)], {}),
    "one key head": ([M.layer(heads=5, kv_heads=1, ff=0)], {}),
    "as many key heads": ([M.layer(heads=3, kv_heads=3, ff=0)], {}),
    "nothing rotates": ([M.layer(rot=0, scaling=None, ff=0)], {}),
    "everything rotates": ([M.layer(dim=16, rot=16, ff=0)], {}),
    "plain frequencies": ([M.layer(scaling=None, ff=0)], {}),
    "feed-forward": ([M.layer(ff=72)], {}),
    "no pairs": ([M.layer()], {"bigram": None}),
    "large factors of the pairs": ([M.layer()], {"bigram": (53, 900001, 10 ** 10 + 7)}),
    "one bucket": ([M.layer()], {"bigram": (1, 2, 3)}),
    "entry of a pass": ([M.layer()], {"loop": (0, 1, 1)}),
}


@BOTH
@pytest.mark.parametrize("name", ALONE)
def test_mechanism_alone(ll, name, dtype):
    layers, more = ALONE[name]
    cfg = M.config(layers, **more)
    w = M.weights(cfg, 11)
    if name == "feed-forward":
        w["l0.ls1"] = w["l0.ls1"] * 0
    toks = M.tokens(cfg, 150, 12)
    want = Expected(cfg, w, toks, dtype)
    m = model(ll, cfg, w, dtype)
    check(feed(m, toks, 150, 0), want, "prompt")
    check(feed(m, toks[:40], 1, 1), want[:40], "decoding")


@BOTH
@pytest.mark.parametrize("loop", [None, (0, 2, 1), (1, 3, 3), (0, 3, 2), (2, 3, 2)])
def test_layer_order_and_loop(ll, loop, dtype):
    cfg = M.config(STACK, loop=loop)
    w, toks = M.weights(cfg, 21), M.tokens(cfg, 90, 22)
    m = model(ll, cfg, w, dtype)
    check(feed(m, toks, cycle(70, 1, 1, 5, 13)), Expected(cfg, w, toks, dtype))


# ---- sizes ---------------------------------------------------------------------------------------------------
SIZES = {
    "odd everywhere": M.config([M.layer(heads=6, kv_heads=3, dim=7, vdim=9, window=5, keep=2, rot=6, ff=33), M.layer(heads=3, kv_heads=1, dim=5, vdim=3, rot=2, ff=21)], width=37, vocab=53,
                               loop=(0, 2, 2)),
    "all ones": M.config([M.layer(heads=1, kv_heads=1, dim=2, vdim=1, window=1, keep=0, rot=2, ff=1)], width=16, vocab=31, bigram=(3, 1, 1), loop=(0, 1, 1)),
    "query heads beyond a block's": M.config([M.layer(heads=38, kv_heads=2, dim=8, vdim=8, window=21)], width=64, vocab=77),
    "sixteen to one": M.config([M.layer(heads=16, kv_heads=1, dim=72, vdim=40, window=50, rot=40, base=1e4)], width=80, vocab=90, loop=(0, 1, 2)),
    "head 128": M.config([M.layer(heads=4, kv_heads=2, dim=128, vdim=128, window=70, keep=9, rot=64, base=1e4)], width=160, vocab=203, loop=(0, 1, 2)),
    "head 192 x 104": M.config([M.layer(heads=2, kv_heads=1, dim=192, vdim=104, window=33, rot=192, base=1e5)], width=72, vocab=99),
    "head 256": M.config([M.layer(heads=2, kv_heads=2, dim=256, vdim=256, window=40, rot=128, base=1e4)], width=64, vocab=99),
    "head 300 x 520": M.config([M.layer(heads=1, kv_heads=1, dim=300, vdim=520, window=30, rot=20)], width=64, vocab=99),
    "head 72 x 300": M.config([M.layer(heads=2, kv_heads=1, dim=72, vdim=300, window=30, rot=20)], width=64, vocab=99),
    "wide": M.config([M.layer(heads=2, kv_heads=1, dim=40, vdim=48, window=30, rot=20, ff=520)], width=1096, vocab=300, loop=(0, 1, 2)),
}


@BOTH
@pytest.mark.parametrize("name", SIZES)
def test_sizes(ll, name, dtype):
    cfg = SIZES[name]
    w, toks = M.weights(cfg, 31), M.tokens(cfg, 100, 32)
    want = Expected(cfg, w, toks, dtype)
    m = model(ll, cfg, w, dtype)
    check(feed(m, toks, 100, 0), want, "prompt")
    check(feed(m, toks[:60], cycle(50, 1, 1, 2, 6), 1), want[:60], "portions")


# ---- portions ------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("sizes", [(2,), (3, 8), (9, 16, 17), (63, 64, 65), (33, 1, 2, 100), (1, 2, 3)])
def test_portions(ll, sizes, dtype):
    cfg = M.config(STACK, loop=(0, 2, 2))
    w, toks = M.weights(cfg, 41), M.tokens(cfg, 203, 42)
    m = model(ll, cfg, w, dtype)
    check(feed(m, toks, cycle(*sizes)), Expected(cfg, w, toks, dtype))


# ---- batches -------------------------------------------------------------------------------------------------
@BOTH
def test_unequal_requests_in_one_step(ll, dtype):
    cfg = M.config(STACK, loop=(1, 2, 2))
    w = M.weights(cfg, 51)
    lens = [70, 1, 33, 16, 5]
    toks = [M.tokens(cfg, n + 12, 52 + i) for i, n in enumerate(lens)]
    want = [Expected(cfg, w, t, dtype) for t in toks]
    m = model(ll, cfg, w, dtype, n_seq=5)
    at = [0] * 5
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


@BOTH
def test_many_sequences_one_token_each(ll, dtype):
    cfg = M.config(STACK, loop=(0, 1, 2))
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
    assert used == 7 + 13, "the first seven stay, and of the widest window (14) what the next token sees"
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
    m.seq_rm(6)
    m.seq_rm(5)
    assert m.kv_used() == 0
    check(feed(m, a[:9], cycle(3, 2), 7), pa[:9], "fewer tokens than are kept")
    assert m.kv_used() == 9
    m.seq_rm(7)
    assert m.kv_used() == 0


def test_interleaved_sequences_scatter_their_cells(ll):
    """sequences that grow in turn hold every other cell; one that ends leaves holes that the next one fills"""
    cfg = M.config(STACK, loop=(0, 1, 2))
    w = M.weights(cfg, 73)
    toks = [M.tokens(cfg, 70, 74 + i) for i in range(3)]
    want = [Expected(cfg, w, t) for t in toks]
    m = model(ll, cfg, w, n_ctx=256, n_seq=2)
    at = [0, 0]
    for step in range(12):
        for s, n in ((0, 1 + step % 5), (1, 1 + step % 3)):
            check(feed(m, toks[s][at[s]:at[s] + n], n, s, at[s]), want[s][at[s]:at[s] + n], f"sequence {s} at {at[s]}")
            at[s] += n
    m.seq_rm(0)
    check(feed(m, toks[2], cycle(20, 1, 4), 2), want[2], "over the holes")
    check(feed(m, toks[1][at[1]:], 9, 1, at[1]), want[1][at[1]:], "its neighbour")


def test_a_full_cache_is_refused_and_survives(ll):
    cfg = M.config([M.layer(window=None)])
    w, toks = M.weights(cfg, 75), M.tokens(cfg, 200, 76)
    want = Expected(cfg, w, toks)
    m = model(ll, cfg, w, n_ctx=256, n_batch=256)
    check(feed(m, toks, 200, 0), want)
    with pytest.raises(b200.load().B200Error):
        feed(m, toks[:100], 100, 1)
    m.seq_rm(0)
    check(feed(m, toks, 100, 1), want)


# ---- edges: one key that stands out, just inside and just outside what a token sees ------------------------------
@BOTH
@pytest.mark.parametrize("window,keep", [(1, 0), (1, 3), (2, 1), (16, 0), (17, 5), (31, 33), (63, 64), (64, 2), (65, 65), (130, 31), (256, 1), (257, 70)])
def test_window_edges_and_kept_tokens(ll, window, keep, dtype):
    cfg, w = M.needle(window, keep)
    for at in sorted({0, max(0, keep - 1), keep, keep + 1, keep + 40}):
        n = max(at, keep) + window + 40
        toks = [t % 59 for t in M.tokens(cfg, n, 82 + at)]
        toks[at] = 59
        want = Expected(cfg, w, toks, dtype)
        edge = at + window                                  # the first token the window alone would not show it to
        m = model(ll, cfg, w, dtype, n_seq=3, n_ctx=1024)
        check(feed(m, toks, n, 0), want, f"prompt, needle at {at}")
        check(feed(m, toks, cycle(max(1, edge - 1), 1, 1, 1), 1), want, f"decoded over the edge, needle at {at}")
        check(feed(m, toks, cycle(max(1, edge - 2), 2, 2, 2, 9, 17), 2), want, f"short portions over the edge, needle at {at}")


@BOTH
def test_far_keys_without_a_mask(ll, dtype):
    """thousands of keys per row: every block and warp of a row's attention goes through several tiles, the needle in any of them"""
    cfg, w = M.needle(None, 0, heads=2, kv_heads=1)
    for at in (0, 1517, 4430):
        toks = [t % 59 for t in M.tokens(cfg, 4500, 88 + at)]
        toks[at] = 59
        want = Expected(cfg, w, toks, dtype)
        if dtype == "float32":
            other = plain(cfg, w).feed([t if i != at else 0 for i, t in enumerate(toks)])
            assert M.error(other[-1:], want.rows[-1:]).max() > 0.05, "the needle must show"
        m = model(ll, cfg, w, dtype, n_ctx=4608, n_batch=4400, n_seq=1)
        check(feed(m, toks, cycle(4400, 1, 1, 7, 8, 1, 30, 5)), want, f"needle at {at}")


def test_pairs_across_portions(ll):
    """a portion's first token is paired with the last one of the portion before, whatever ran in between"""
    cfg = M.config([M.layer(ff=0)])
    w, a, b = M.weights(cfg, 85), M.tokens(cfg, 30, 86), M.tokens(cfg, 30, 87)
    wa, wb = Expected(cfg, w, a), Expected(cfg, w, b)
    m = model(ll, cfg, w, n_seq=2)
    for i in range(0, 30, 3):
        check(feed(m, a[i:i + 3], 3, 0, i), wa[i:i + 3])
        check(feed(m, b[i:i + 3], 1, 1, i), wb[i:i + 3])
    m.seq_rm(0)
    check(feed(m, b[:4], 2, 0), wb[:4], "a slot's first token has none before it")


def test_sinks_and_first_tokens(ll):
    """large sinks dominate the first tokens, whose windows are nearly empty"""
    cfg = M.config([M.layer(window=12, ff=0)])
    w, toks = M.weights(cfg, 95), M.tokens(cfg, 20, 96)
    w["l0.norm1b.b"] = w["l0.norm1b.b"] * 0
    w["l0.norm1b"] = w["l0.norm1b"] * 0 + 1
    for sinks in (-20.0, 0.0, 6.0):
        w["l0.mix.sink"] = np.array([sinks, 1.0, -sinks, 0.5], np.float32)
        want = Expected(cfg, w, toks)
        m = model(ll, cfg, w)
        check(feed(m, toks, 20, 0), want, f"sink {sinks}, prompt")
        check(feed(m, toks, 1, 1), want, f"sink {sinks}, decoding")


def test_far_positions(ll):
    """angles and windows thousands of tokens into a sequence"""
    cfg = M.config([M.layer(dim=16, window=20, keep=2, rot=16, base=1e4, ff=0)])
    w, toks = M.weights(cfg, 97), M.tokens(cfg, 5000, 98)
    want = Expected(cfg, w, toks)
    m = model(ll, cfg, w, n_ctx=1024, n_batch=700)
    check(feed(m, toks, cycle(700, 650, 1, 1, 3)), want)


# ---- long decoding, generation, folders ----------------------------------------------------------------------------
@BOTH
def test_long_decoding(ll, dtype):
    cfg = M.config(STACK, loop=(0, 3, 2))
    w, toks = M.weights(cfg, 101), M.tokens(cfg, 420, 102)
    m = model(ll, cfg, w, dtype, n_ctx=256, n_batch=64, n_seq=1)   # fewer cells than tokens: windows slide over used cells
    check(feed(m, toks, cycle(60, *[1] * 360)), Expected(cfg, w, toks, dtype))


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
        want = Expected(cfg, w, toks, dtype)
        for step, rows in ((0, [46, 3]), (2, [49]), (3, [4])):
            check(np.fromfile(tmp_path / f"{step}.f32", np.float32).reshape(len(rows), -1), want[rows], f"step {step}")


def test_the_stream_after_a_layer_run(ll):
    """the residual stream itself, not only the logits behind the last norm"""
    cfg = M.config(STACK[:2] + [M.layer()], loop=(0, 2, 2))
    w, toks = M.weights(cfg, 125), M.tokens(cfg, 33, 126)
    p = plain(cfg, w)
    p.feed(toks)
    m = model(ll, cfg, w)
    feed(m, toks, 33)
    got = m.read_node("l_out", 33 * 48).reshape(33, 48)
    assert np.abs(got - p.residuals[-1]).max() < 2e-5 * np.abs(p.residuals[-1]).max()


def test_missing_and_misshapen_tensors_are_refused(ll):
    mod = b200.load()
    cfg = M.config([M.layer(), M.layer()], loop=(0, 1, 2))
    w = M.weights(cfg, 131)
    m = ll.Model(cfg, 256, 32, dtype="float32")
    for name, bad in (("l1.mix.o", w["l1.mix.o"][:-1]), ("loop.in", w["loop.in"][:, :48]), ("bigram", w["bigram"][:-1]), ("l0.mlp.gate", w["l0.mlp.up"][:-2])):
        with pytest.raises(mod.B200Error):
            m.set_tensors({name: bad})
    with pytest.raises(mod.B200Error):
        m.set_tensors({"l7.norm1": w["l0.norm1"]})
    m.set_tensors({k: v for k, v in w.items() if k != "l1.mlp.gate"})
    with pytest.raises(mod.B200Error, match="l1.mlp.gate"):
        m.decode_seqs([1], [0], [0], [0])
    m.set_tensors({"l1.mlp.gate": w["l1.mlp.gate"]})        # its rows go between those of up, which stay
    toks = M.tokens(cfg, 10, 132)
    m.kv_clear()
    check(feed(m, toks, 10), Expected(cfg, w, toks))
