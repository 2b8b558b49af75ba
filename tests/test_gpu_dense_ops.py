"""The ops of decoders with dense weights, one node at a time through the plug-in face, against plain float64 arithmetic."""
import ctypes as C

import numpy as np
import pytest

import b200
import ggml_plugin as gp
import plain_decoder as P
import rukusun_models as M

pytestmark = pytest.mark.gpu

DENSE_MM, RMS_NORM_W, TAKE_ROWS, GLA = 0x4210, 0x4211, 0x4212, 0x4213
LATENT_DECODE = 0x4216


@pytest.fixture(scope="module")
def lib():
    return gp.load_backend(b200.load().LIB_PATH)


@pytest.fixture
def sess(lib):
    s = gp.Session(*lib, buffer_bytes=1 << 28)
    yield s
    s.close()


def put(s, arr, ty=gp.F32):
    """rows of arr (last dimension first in ne) as a tensor of the type"""
    arr = np.ascontiguousarray(arr)
    t = s.new_tensor(ty, list(arr.shape[::-1]))
    if ty == gp.BF16:
        arr = (M.bf16(arr).view(np.uint32) >> 16).astype(np.uint16)
    s.set(t, arr.astype({gp.F32: np.float32, gp.I32: np.int32}.get(ty, arr.dtype), copy=False))
    return t


def get(s, t):
    n = t.ne[0] * t.ne[1] * t.ne[2]
    if t.type == gp.BF16:
        return (s.get(t, np.uint16, n).astype(np.uint32) << 16).view(np.float32).reshape(t.ne[1], t.ne[0])
    return s.get(t, np.float32, n).reshape(t.ne[1], t.ne[0])


def node(s, op, ty, ne, srcs, ints=(), floats=()):
    t = s.new_tensor(ty, ne)
    t.op = op
    for i, x in enumerate(srcs):
        if x is not None:
            t.src[i] = C.pointer(x)
    for i, v in ints:
        t.op_params[i] = v
    for i, v in floats:
        t.op_params[i] = int(np.float32(v).view(np.int32))
    return t


@pytest.mark.parametrize("wt,xt,yt", [(gp.BF16, gp.BF16, gp.F32), (gp.BF16, gp.BF16, gp.BF16), (gp.BF16, gp.F32, gp.F32), (gp.F32, gp.F32, gp.F32)],
                         ids=["bf16", "bf16-out-bf16", "bf16-f32", "f32"])
@pytest.mark.parametrize("n,k,m", [(5, 8, 1), (130, 40, 3), (96, 264, 7), (33, 20, 16), (257, 72, 17), (64, 64, 64), (300, 136, 70), (129, 200, 131), (520, 1000, 300), (70, 37, 90)])
def test_dense_mat_mul(sess, n, k, m, wt, xt, yt):
    rng = np.random.default_rng(n + k + m)
    w, x, add = M.bf16(rng.standard_normal((n, k))), M.bf16(rng.standard_normal((m, k))), rng.standard_normal((m, n)).astype(np.float32)
    tw, tx, ta = put(sess, w, wt), put(sess, x, xt), put(sess, add)
    plain = x.astype(np.float64) @ w.T.astype(np.float64)
    scale = np.abs(x.astype(np.float64)) @ np.abs(w.T.astype(np.float64)) + 1.0
    for act, addend in ((0, None), (1, None), (0, ta), (1, ta)):
        y = node(sess, DENSE_MM, yt, [n, m], [tw, tx, addend], ints=[(0, act)])
        assert sess.compute([y]) == 0, sess.last_error()
        want = (P.gelu_tanh(plain) if act else plain) + (add if addend is not None else 0.0)
        got = get(sess, y)
        assert np.allclose(got, want, rtol=2 ** -8, atol=1e-4 * scale.max()) if yt == gp.BF16 else (np.abs(got - want) <= 2e-6 * scale).all()


@pytest.mark.parametrize("m", [255, 513, 2048])
def test_wide_tiles(sess, m):
    """enough tiles that the 256-column form is taken, ragged on both sides"""
    n, k = 4096 + 60, 264
    rng = np.random.default_rng(m)
    w, x = M.bf16(rng.standard_normal((n, k))), M.bf16(rng.standard_normal((m, k)))
    y = node(sess, DENSE_MM, gp.F32, [n, m], [put(sess, w, gp.BF16), put(sess, x, gp.BF16)])
    assert sess.compute([y]) == 0, sess.last_error()
    want = x.astype(np.float64) @ w.T.astype(np.float64)
    assert np.abs(get(sess, y) - want).max() < 1e-4


@pytest.mark.parametrize("wt", [gp.BF16, gp.F32])
@pytest.mark.parametrize("n,k,m", [(50, 48, 1), (7, 37, 2), (300, 512, 5), (64, 1028, 16)])
def test_norm_inside_the_mat_mul(sess, n, k, m, wt):
    rng = np.random.default_rng(k)
    w, x, g = M.bf16(rng.standard_normal((n, k))), rng.standard_normal((m, k)).astype(np.float32), (1 + 0.3 * rng.standard_normal(k)).astype(np.float32)
    y = node(sess, DENSE_MM, gp.F32, [n, m], [put(sess, w, wt), put(sess, x), None, put(sess, g)], floats=[(1, 1e-3)])
    assert sess.compute([y]) == 0, sess.last_error()
    h = P.rms_norm_plain(x.astype(np.float64), g.astype(np.float64), 1e-3)
    assert np.abs(get(sess, y) - h @ w.T).max() < 2e-6 * (np.abs(h) @ np.abs(w.T)).max()
    t = node(sess, DENSE_MM, gp.F32, [n, 17], [put(sess, w, wt), put(sess, np.zeros((17, k))), None, put(sess, g)])
    assert not sess.supports(t)          # only while there are few rows


@pytest.mark.parametrize("yt", [gp.F32, gp.BF16])
@pytest.mark.parametrize("k,m", [(37, 3), (512, 40), (9000, 2)])
def test_norm_and_rows(sess, k, m, yt):
    rng = np.random.default_rng(k)
    x, g = rng.standard_normal((m, k)).astype(np.float32), rng.standard_normal(k).astype(np.float32)
    tx = put(sess, x)
    y = node(sess, RMS_NORM_W, yt, [k, m], [tx, put(sess, g)], floats=[(0, 1e-2)])
    ids = rng.integers(0, m, 9)
    r = node(sess, TAKE_ROWS, yt, [k, 9], [tx, put(sess, ids, gp.I32)], floats=[(0, 3.5)])
    assert sess.compute([y, r]) == 0, sess.last_error()
    rtol = 2 ** -8 if yt == gp.BF16 else 1e-6
    assert np.allclose(get(sess, y), P.rms_norm_plain(x.astype(np.float64), g.astype(np.float64), 1e-2), rtol=rtol, atol=1e-6)
    assert np.allclose(get(sess, r), x[ids] * 3.5, rtol=rtol, atol=1e-6)


def test_a_row_outside_the_table_is_reported(sess):
    y = node(sess, TAKE_ROWS, gp.F32, [8, 2], [put(sess, np.ones((4, 8))), put(sess, np.array([1, 4]), gp.I32)], floats=[(0, 1.0)])
    assert sess.compute([y]) == 0
    assert b200.load().kernel_error() == 1 and (get(sess, y)[0] == 1).all()


@pytest.mark.parametrize("H,d,e,tau", [(2, 16, 8, 4.0), (3, 130, 20, 16.0), (1, 260, 300, 0.5), (2, 64, 128, 1.0)])
@pytest.mark.parametrize("rows", [[1, 1, 1], [5, 16], [17, 1, 64], [65, 130, 2]])
def test_gla_over_segments(sess, H, d, e, tau, rows):
    """sequences of different lengths in one node, some going on from a state, in both forms"""
    rng = np.random.default_rng(sum(rows) + d)
    R, n, P_ = 4, sum(rows), 2 * H * d + 2 * H * e + 4
    proj = rng.standard_normal((n, P_)).astype(np.float32)
    a2, bias, norm = M.bf16(rng.standard_normal((H * d, R))), rng.uniform(-3, 4, H * d).astype(np.float32), rng.standard_normal(e).astype(np.float32)
    state = rng.standard_normal((len(rows) + 1, H, d, e)).astype(np.float32)
    seg, at = [], 0
    for i, r in enumerate(rows):
        seg.append([at, r, len(rows) - i, i % 2, 0, 0, 0, 0])     # slots in reverse, every other one fresh
        at += r
    lib_floats = 1 << 22
    ts, tseg = put(sess, state.reshape(len(rows) + 1, -1)), put(sess, np.array(seg), gp.I32)
    for scratch in ([None] if max(rows) <= 16 else [put(sess, np.zeros(lib_floats, np.float32)), None]):
        sess.set(ts, state)
        y = node(sess, GLA, gp.F32, [H * e, n], [put(sess, proj), put(sess, a2, gp.BF16), put(sess, bias), put(sess, norm), ts, tseg, scratch],
                 ints=[(0, H), (1, d), (2, e), (3, 0), (4, H * d), (5, 2 * H * d), (6, 2 * H * d + H * e), (7, 2 * H * d + 2 * H * e), (11, max(rows)), (12, R)],
                 floats=[(8, d ** -0.5), (9, 1 / tau), (10, 1e-4)])
        assert sess.compute([y]) == 0, sess.last_error()
        got, after = get(sess, y), sess.get(ts, np.float32, state.size).reshape(state.shape)
        assert np.array_equal(after[0], state[0]), "a slot no sequence has"
        x = proj.astype(np.float64)
        for r0, r, slot, fresh, *_ in seg:
            p = x[r0:r0 + r]
            q, k = p[:, :H * d].reshape(r, H, d) * d ** -0.5, p[:, H * d:2 * H * d].reshape(r, H, d)
            v, g = p[:, 2 * H * d:2 * H * d + H * e].reshape(r, H, e), p[:, 2 * H * d + H * e:2 * H * d + 2 * H * e]
            al = P.gla_decay((p[:, -R:] @ a2.T.astype(np.float64) + bias).reshape(r, H, d), tau)
            o, S = P.gla_recurrence(q, k, v, al, np.zeros((H, d, e)) if fresh else state[slot].astype(np.float64))
            want = P.rms_norm_plain(o, norm, 1e-4).reshape(r, H * e) * P.silu(g)
            assert np.abs(got[r0:r0 + r] - want).max() < 1e-4 and np.abs(after[slot] - S).max() < 1e-5 * max(1.0, np.abs(S).max())


def test_malformed_nodes_are_refused(sess):
    w, x = put(sess, np.zeros((8, 16)), gp.BF16), put(sess, np.zeros((3, 16)))
    assert sess.supports(node(sess, DENSE_MM, gp.F32, [8, 3], [w, x]))
    assert not sess.supports(node(sess, DENSE_MM, gp.F32, [9, 3], [w, x]))
    assert not sess.supports(node(sess, DENSE_MM, gp.F32, [8, 3], [w, put(sess, np.zeros((3, 17)))]))
    assert not sess.supports(node(sess, DENSE_MM, gp.F32, [8, 3], [w, x], ints=[(0, 7)]))
    assert not sess.supports(node(sess, DENSE_MM, gp.F32, [8, 3], [w, None]))
    assert not sess.supports(node(sess, RMS_NORM_W, gp.F32, [16, 3], [x, put(sess, np.zeros(15))]))
    assert not sess.supports(node(sess, GLA, gp.F32, [4, 3], [x, w, None, None], ints=[(0, 1), (1, 2), (2, 4), (12, 1)]))
    assert not sess.supports(node(sess, LATENT_DECODE, gp.F32, [4, 1, 3], [x, None, w], ints=[(0, 1), (1, 2), (2, 2), (3, 2), (4, 2)]))
    bad = node(sess, DENSE_MM, gp.F32, [9, 3], [w, x])
    assert sess.compute([bad]) != 0 and "dense" in sess.last_error()


def test_a_segment_outside_the_step_is_reported(sess):
    """a slot the state has not, rows the step has not: skipped and reported, the rest of the node unharmed"""
    H, d, e, R, n = 1, 8, 8, 1, 40
    rng = np.random.default_rng(1)
    proj, state = rng.standard_normal((n, 2 * d + 2 * e + R)).astype(np.float32), np.zeros((2, d * e), np.float32)
    ts = put(sess, state)
    srcs = [put(sess, proj), put(sess, np.ones((d, R)), gp.BF16), put(sess, np.ones(d)), put(sess, np.ones(e)), ts]
    for scratch in (None, put(sess, np.zeros(1 << 18, np.float32))):
        for bad in ([20, 20, 2, 1, 0, 0, 0, 0], [20, 21, 1, 1, 0, 0, 0, 0], [-1, 20, 1, 1, 0, 0, 0, 0]):
            sess.set(ts, state)
            y = node(sess, GLA, gp.F32, [H * e, n], srcs + [put(sess, np.array([[0, 20, 0, 1, 0, 0, 0, 0], bad]), gp.I32), scratch],
                     ints=[(0, H), (1, d), (2, e), (3, 0), (4, d), (5, 2 * d), (6, 2 * d + e), (7, 2 * d + 2 * e), (11, 20), (12, R)], floats=[(8, 1.0), (9, 1.0), (10, 1e-5)])
            assert sess.compute([y]) == 0, sess.last_error()
            assert b200.load().kernel_error() == 6
            after = sess.get(ts, np.float32, 2 * d * e).reshape(2, -1)
            assert after[0].any() and not after[1].any() and np.isfinite(get(sess, y)[:20]).all()
