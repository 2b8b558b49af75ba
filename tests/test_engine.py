"""The serving loop and the trace replay on the host: a stand-in context that only counts, no GPU."""
import importlib

import numpy as np
import pytest

import b200


@pytest.fixture(scope="module")
def engine():
    b200.load()
    return importlib.import_module("llama_rust_b200.engine")


class Counting:
    """next token = (sum of the sequence's tokens so far) % vocab; checks what a context would insist on"""
    n_vocab = 50

    def __init__(self, n_batch, n_seq):
        self.n_batch, self.n_seq, self.kept, self.calls = n_batch, n_seq, {}, []

    def decode_seqs(self, tokens, pos, seq_ids, out_rows, logits=True, argmax=False):
        assert 0 < len(tokens) <= self.n_batch and len(tokens) == len(pos) == len(seq_ids)
        self.calls.append(list(zip(seq_ids, pos)))
        seen, sums = [], []
        for t, p, s in zip(tokens, pos, seq_ids):
            if not seen or seen[-1] != s:
                assert s not in seen, "a sequence's rows stand together"
                seen.append(s)
            mine = self.kept.setdefault(s, [])
            assert p == len(mine)
            mine.append(t)
            sums.append(sum(mine) % self.n_vocab)
        assert len(self.kept) <= self.n_seq
        picked = np.array([sums[r] for r in out_rows], dtype=np.int32)
        lg = np.zeros((len(out_rows), self.n_vocab), np.float32)
        lg[np.arange(len(out_rows)), picked] = 1.0
        return (lg if logits else None), (picked if argmax else None)

    def seq_rm(self, s):
        del self.kept[s]


def alone(prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(sum(t) % Counting.n_vocab)
    return t[len(prompt):]


@pytest.mark.parametrize("n_batch,n_seq,portion", [(64, 8, None), (7, 3, None), (16, 2, 4), (5, 8, 2), (1, 1, None)])
def test_every_request_is_served_as_if_alone(engine, n_batch, n_seq, portion):
    rng = np.random.default_rng(n_batch)
    prompts = [rng.integers(0, 50, n).tolist() for n in (3, 11, 1, 8, 20, 2)]
    ctx = Counting(n_batch, n_seq)
    out = engine.generate(ctx, prompts, 6, max_seqs=n_seq, portion=portion)
    assert out == [alone(p, 6) for p in prompts]
    assert not ctx.kept and max(len(c) for c in ctx.calls) <= n_batch


def test_stop_token_and_mixed_steps(engine):
    ctx = Counting(8, 4)
    e = engine.Engine(ctx, 4, portion=4)
    e.submit(engine.Request("a", [1, 2], 9, stop=[6]))      # 3, 6
    e.submit(engine.Request("b", list(range(12)), 2))
    out = e.run()
    assert out["a"] == [3, 6] and out["b"] == alone(range(12), 2)
    assert any({"a", "b"} == {r for r, _ in step} for step in e.steps)
    with pytest.raises(ValueError):
        e.submit(engine.Request("c", [], 1))


def test_replay_keeps_order_across_decode_calls(engine):
    ctx = Counting(4, 2)
    r = engine.Replay(ctx)
    got = r.step([("x", [1, 2, 3, 4, 5, 6, 7], [6, 0, 4])])
    assert got.argmax(1).tolist() == [28, 1, 15]
    assert r.step([("x", [1], [])]).shape == (0, 50)
    r.end("x")
    assert not ctx.kept and r.step([("y", [9], [0])]).argmax(1).tolist() == [9]


def test_configurations_that_describe_no_model_are_refused():
    import rukusun_models as M
    mod = b200.load()
    ll = importlib.import_module("llama_rust_b200.llama")

    def refused(change):
        cfg = M.config([M.gla(), M.latent()], loop=(0, 1, 2))
        change(cfg)
        with pytest.raises(mod.B200Error) as e:
            ll.Model(cfg, 256, 32)
        return str(e.value)

    assert "architecture" in refused(lambda c: c.update(architecture="Other"))
    assert "heads" in refused(lambda c: c["layers"][0]["mixer"].pop("heads"))
    assert "not known" in refused(lambda c: c["layers"][0].update(type="other"))
    assert "loop" in refused(lambda c: c["loop"].update(stop=3))
    assert "tau" in refused(lambda c: c["layers"][0]["mixer"].update(tau=0))
    assert "dense" in refused(lambda c: c["layers"][1]["mlp"].update(kind="other"))
    assert "rotated" in refused(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7))


def test_lenolix_configurations_that_describe_no_model_are_refused():
    import lenolix_models as M
    mod = b200.load()
    ll = importlib.import_module("llama_rust_b200.llama")

    def refused(change):
        cfg = M.config([M.layer(), M.layer()], loop=(0, 1, 2))
        change(cfg)
        with pytest.raises(mod.B200Error) as e:
            ll.Model(cfg, 256, 32)
        return str(e.value)

    mixer = lambda c: c["layers"][1]["mixer"]  # noqa: E731
    assert "kv_heads" in refused(lambda c: mixer(c).pop("kv_heads"))
    assert "multiple of kv_heads" in refused(lambda c: mixer(c).update(kv_heads=3))
    assert "not known" in refused(lambda c: c["layers"][0].update(type="gla"))
    assert "rotated" in refused(lambda c: mixer(c)["rot"].update(dims=7))
    assert "rotated" in refused(lambda c: mixer(c)["rot"].update(dims=22))
    assert "scaling" in refused(lambda c: mixer(c)["rot"]["scaling"].update(factor=0))
    assert "mask" in refused(lambda c: mixer(c)["mask"].update(size=0))
    assert "keep_first" in refused(lambda c: mixer(c)["mask"].update(keep_first=-1))
    assert "limit" in refused(lambda c: c["layers"][0]["mlp"].pop("limit"))
    assert "dense" in refused(lambda c: c["layers"][0]["mlp"].update(kind="other"))
    assert "buckets" in refused(lambda c: c["embedding"]["bigram"].update(buckets=0))
    assert "bigram" in refused(lambda c: c["embedding"]["bigram"].update(mul_cur=1.5))
    assert "loop" in refused(lambda c: c["loop"].update(stop=3))
