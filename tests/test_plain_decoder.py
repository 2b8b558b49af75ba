"""The plain decoder the GPU tests compare with: its mechanisms against closed forms, its two ways of feeding a sequence against
each other, and that the models the tests use make a mistake in any mechanism show (the mistake is planted in the plain decoder)."""
import copy

import numpy as np
import pytest

import plain_decoder as P
import rukusun_models as M


def test_norms_gate_and_activation():
    x = np.array([[3.0, -4.0]])
    assert np.allclose(P.rms(x, 0.0), x / np.sqrt(12.5))
    assert np.allclose(P.rms_norm_around_zero(x, np.array([0.0, 1.0]), 0.5), x / np.sqrt(13.0) * [1.0, 2.0])
    z = np.linspace(-30, 30, 7)
    assert np.allclose(P.sigmoid(z), 1 / (1 + np.exp(-z))) and np.allclose(P.silu(z), z / (1 + np.exp(-z)))
    assert np.allclose(P.gelu_tanh(np.array([0.0, 1.0])), [0.0, 0.8411919906], atol=1e-9)


def test_rotation_turns_pairs_and_keeps_relative_angles():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal(8), rng.standard_normal(8)
    a = P.rotate_interleaved(q, 13, 100.0, 6) @ P.rotate_interleaved(k, 5, 100.0, 6)
    b = P.rotate_interleaved(q, 1008, 100.0, 6) @ P.rotate_interleaved(k, 1000, 100.0, 6)
    assert np.isclose(a, b) and np.array_equal(P.rotate_interleaved(q, 7, 100.0, 6)[6:], q[6:])
    one = P.rotate_interleaved(np.array([1.0, 0.0]), 2, 10.0, 2)
    assert np.allclose(one, [np.cos(2.0), np.sin(2.0)])


def test_window_and_sink():
    assert list(P.window_keys(5, 3)) == [3, 4, 5] and list(P.window_keys(1, 3)) == [0, 1] and list(P.window_keys(4, None)) == [0, 1, 2, 3, 4]
    w = P.softmax_with_sink(np.array([1.0, 2.0]), 0.5)
    e = np.exp([1.0, 2.0])
    assert np.allclose(w, e / (e.sum() + np.exp(0.5)))


def test_gla_recurrence_is_the_weighted_sum_over_the_past():
    rng = np.random.default_rng(1)
    T, H, d, e = 7, 2, 3, 4
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, H, d)), rng.standard_normal((T, H, e))
    al = P.gla_decay(rng.standard_normal((T, H, d)) * 3, 2.0)
    out, S = P.gla_recurrence(q, k, v, al, np.zeros((H, d, e)))
    for t in range(T):
        for h in range(H):
            want = sum((q[t, h] * k[j, h] * np.prod(al[j + 1:t + 1, h], axis=0)).sum() * v[j, h] for j in range(t + 1))
            assert np.allclose(out[t, h], want)


@pytest.mark.parametrize("layers,loop", [([M.gla(), M.latent()], None), ([M.latent(window=4), M.gla(ff=0)], (0, 2, 2))])
def test_token_by_token_is_the_whole_prompt(layers, loop):
    cfg = M.config(layers, loop=loop)
    w, toks = M.weights(cfg, 3), M.tokens(cfg, 23, 4)
    whole = P.Plain(cfg, w).feed(toks)
    p = P.Plain(cfg, w)
    one = np.concatenate([p.feed([t]) for t in toks])
    assert np.allclose(whole, one)


def planted(cfg, w, toks, change):
    c, v = copy.deepcopy(cfg), dict(w)
    change(c, v)
    return M.error(P.Plain(c, v).feed(toks), P.Plain(cfg, w).feed(toks)).max()


@pytest.mark.parametrize("change", [
    lambda c, w: c["layers"][1]["mixer"]["mask"].update(size=10),
    lambda c, w: c["layers"][1]["mixer"]["mask"].update(size=8),
    lambda c, w: c["layers"][1]["mixer"]["rot"].update(base=1100.0),
    lambda c, w: c["layers"][1]["mixer"].update(scale=0.15),
    lambda c, w: w.update({"l1.mix.sink": np.full(3, -30.0)}),
    lambda c, w: w.update({"l1.mix.dkv.norm": np.ones(40)}),
    lambda c, w: c["layers"][0]["mixer"].update(tau=4.2),
    lambda c, w: w.update({"l0.mix.a2.b": w["l0.mix.a2.b"] * 0}),
    lambda c, w: w.update({"l0.mix.norm": np.ones(12)}),
    lambda c, w: c["norm"].update(eps=1e-3),
    lambda c, w: c["embedding"].update(scale=5.5),
    lambda c, w: w.update({"loop.step": w["loop.step"][::-1]}),
    lambda c, w: c["loop"].update(times=1),
])
def test_a_planted_mistake_shows(change):
    cfg = M.config([M.gla(), M.latent()], loop=(0, 2, 2))
    w, toks = M.weights(cfg, 5), M.tokens(cfg, 40, 6)
    assert planted(cfg, w, toks, change) > 1e-3
