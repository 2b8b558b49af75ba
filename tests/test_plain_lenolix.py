"""The plain restatement of Lenolix the GPU tests compare with: its mechanisms against closed forms, its ways of feeding a sequence
against each other, and that the tests' models make a mistake in any mechanism show (the mistake is planted in the plain decoder)."""
import copy

import numpy as np
import pytest

import lenolix_models as M
import plain_lenolix as L


def test_norm_gate_and_pairs():
    x = np.array([[1.0, 3.0, 8.0]])
    assert np.allclose(L.layer_norm(x, np.array([1.0, 2.0, 1.0]), np.array([0.0, 0.0, 5.0]), 1.0), [[-3 / np.sqrt(29 / 3), -2 / np.sqrt(29 / 3), 5 + 4 / np.sqrt(29 / 3)]])
    s = lambda z: 1 / (1 + np.exp(-z))  # noqa: E731
    assert np.allclose(L.gated(np.array([9.0, -9.0, 1.0]), np.array([0.5, 9.0, -9.0]), 2.0), [2 * s(3.404) * 1.5, -9 * s(-9 * 1.702) * 3, -s(1.702)])
    spec = {"buckets": 7, "mul_prev": 3, "mul_cur": 2}
    assert [L.pair_row(None, 5, spec), L.pair_row(4, 5, spec), L.pair_row(0, 0, spec)] == [7, 1, 0]


def test_frequencies_are_kept_ramped_and_stretched():
    rot = {"base": 500.0, "dims": 8, "scaling": M.RAMP}
    f, plain = L.frequencies(rot), L.frequencies(dict(rot, scaling=None))
    wave = 2 * np.pi / plain
    assert wave[0] < 16 and 16 < wave[1] < 64 and wave[2] > 64
    s = (64 / wave[1] - 1) / 3
    assert np.isclose(f[0], plain[0]) and np.allclose(f[2:], plain[2:] / 4) and np.isclose(f[1], (1 - s) * plain[1] / 4 + s * plain[1])


def test_rotation_turns_halves_and_keeps_relative_angles():
    rng = np.random.default_rng(0)
    rot = {"base": 100.0, "dims": 6}
    q, k = rng.standard_normal(8), rng.standard_normal(8)
    a = L.rotate_halves(q, 13, rot)[:6] @ L.rotate_halves(k, 5, rot)[:6]
    b = L.rotate_halves(q, 1008, rot)[:6] @ L.rotate_halves(k, 1000, rot)[:6]
    assert np.isclose(a, b) and np.array_equal(L.rotate_halves(q, 7, rot)[6:], q[6:])
    one = L.rotate_halves(np.array([1.0, 5.0, 0.0, 0.0]), 2, {"base": 10.0, "dims": 4})
    assert np.allclose(one, [np.cos(2.0), 5 * np.cos(2 * 10 ** -0.5), np.sin(2.0), 5 * np.sin(2 * 10 ** -0.5)])


def test_visible_positions():
    m = {"size": 3, "keep_first": 2}
    assert [L.visible(i, m) for i in (0, 1, 3, 4, 6)] == [[0], [0, 1], [0, 1, 2, 3], [0, 1, 2, 3, 4], [0, 1, 4, 5, 6]]
    assert list(L.visible(2, None)) == [0, 1, 2] and L.visible(5, {"size": 1}) == [5]


@pytest.mark.parametrize("loop", [None, (0, 2, 2), (1, 2, 3)])
def test_token_by_token_is_the_whole_prompt(loop):
    cfg = M.config([M.layer(), M.layer(kv_heads=4, window=4, ff=0)], loop=loop)
    w, toks = M.weights(cfg, 3), M.tokens(cfg, 23, 4)
    p = L.Plain(cfg, w)
    assert np.allclose(L.Plain(cfg, w).feed(toks), np.concatenate([p.feed([t]) for t in toks]))


def planted(cfg, w, toks, change):
    c, v = copy.deepcopy(cfg), dict(w)
    change(c, v)
    return M.error(L.Plain(c, v).feed(toks), L.Plain(cfg, w).feed(toks)).max()


@pytest.mark.parametrize("change", [
    lambda c, w: c["layers"][1]["mixer"]["mask"].update(size=10),
    lambda c, w: c["layers"][1]["mixer"]["mask"].update(size=8),
    lambda c, w: c["layers"][1]["mixer"]["mask"].update(keep_first=4),
    lambda c, w: c["layers"][1]["mixer"]["mask"].update(keep_first=2),
    lambda c, w: c["layers"][1]["mixer"]["rot"].update(base=550.0),
    lambda c, w: c["layers"][1]["mixer"]["rot"].update(scaling=None),
    lambda c, w: c["layers"][1]["mixer"]["rot"].update(scaling=dict(M.RAMP, high=5.0)),
    lambda c, w: c["layers"][1]["mixer"].update(scale=0.25),
    lambda c, w: w.update({"l1.mix.sink": np.full(4, -30.0)}),
    lambda c, w: c["layers"][0]["mlp"].update(limit=1.6),
    lambda c, w: w.update({"l0.norm1b.b": np.zeros(48)}),
    lambda c, w: w.update({"l0.norm2.b": np.zeros(48)}),
    lambda c, w: w.update({"l1.ls1": np.ones(48)}),
    lambda c, w: w.update({"l0.ls2": np.ones(48)}),
    lambda c, w: c["norm"].update(eps=3e-3),
    lambda c, w: c["embedding"].update(scale=5.5),
    lambda c, w: c["embedding"].update(bigram=None),
    lambda c, w: c["embedding"]["bigram"].update(mul_prev=3, mul_cur=5),
    lambda c, w: w.update({"loop.step": w["loop.step"][::-1]}),
    lambda c, w: w.update({"loop.in": w["loop.in"][:, list(range(48, 96)) + list(range(48))]}),
    lambda c, w: c["loop"].update(times=1),
])
def test_a_planted_mistake_shows(change):
    cfg = M.config([M.layer(), M.layer()], loop=(0, 2, 2))
    w, toks = M.weights(cfg, 5), M.tokens(cfg, 40, 6)
    assert planted(cfg, w, toks, change) > 1e-3


@pytest.mark.parametrize("window,keep", [(1, 0), (2, 1), (17, 3), (64, 5), (33, 64)])
def test_the_needle_shows(window, keep):
    cfg, w = M.needle(window, keep)
    for at in (0, max(0, keep - 1), keep, keep + 7):
        toks = [t % 59 for t in M.tokens(cfg, window + at + 12, 82 + at)]
        toks[at] = 59
        p = L.Plain(cfg, w).feed(toks)
        seen = planted(cfg, w, toks, lambda c, v: c["layers"][0]["mixer"]["mask"].update(size=window + 1))
        assert seen > 0.1 if at >= keep else seen < 1e-2, (at, seen)
        if at < keep:
            assert planted(cfg, w, toks, lambda c, v: c["layers"][0]["mixer"]["mask"].update(keep_first=at)) > 0.1
        assert np.isfinite(p).all()
