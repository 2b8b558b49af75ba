"""The ops of decoders with dense weights, one node at a time through the plug-in face, against plain float64 arithmetic."""
import ctypes as C

import numpy as np
import pytest

import b200
import ggml_plugin as gp
import plain_decoder as P
import plain_lenolix as L
import rukusun_models as M

pytestmark = pytest.mark.gpu

DENSE_MM, RMS_NORM_W, TAKE_ROWS, GLA = 0x4210, 0x4211, 0x4212, 0x4213
LATENT_DECODE = 0x4216
PAIR_EMBED, LAYER_NORM_W, NORM_SUM, GROUPED_STORE, GROUPED_DECODE, GROUPED_ATTN = range(0x4219, 0x421f)


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


def strided(s, t, ne0, ne1, nb1, offset=0):
    """rows of ne0 elements, nb1 bytes apart, inside t"""
    v = s.new_tensor(t.type, [1])
    v.ne[0], v.ne[1], v.ne[2], v.ne[3] = ne0, ne1, 1, 1
    v.nb[0], v.nb[1], v.nb[2], v.nb[3] = t.nb[0], nb1, nb1 * ne1, nb1 * ne1
    v.data = t.data + offset
    return v


TYPES = pytest.mark.parametrize("wt,xt,yt", [(gp.BF16, gp.BF16, gp.F32), (gp.BF16, gp.BF16, gp.BF16), (gp.BF16, gp.F32, gp.F32), (gp.F32, gp.F32, gp.F32)],
                                ids=["bf16", "bf16-out-bf16", "bf16-f32", "f32"])


@TYPES
@pytest.mark.parametrize("n,k,m", [(2, 8, 1), (6, 37, 3), (130, 264, 16), (96, 40, 70), (322, 136, 300), (4096, 64, 600)])
def test_clamped_gate_over_pairs_of_rows(sess, n, k, m, wt, xt, yt):
    rng = np.random.default_rng(n + k + m)
    w, x, bias = M.bf16(rng.standard_normal((n, k))), M.bf16(rng.standard_normal((m, k))), rng.standard_normal(n).astype(np.float32)
    tw, tx, tb = put(sess, w, wt), put(sess, x, xt), put(sess, bias)
    plain = x.astype(np.float64) @ w.T.astype(np.float64)
    for b in (None, tb):
        for limit, alpha in ((3.0, 1.702), (0.5, 1.0)):
            y = node(sess, DENSE_MM, yt, [n // 2, m], [tw, tx, None, None, b], ints=[(0, 2)], floats=[(2, limit), (3, alpha)])
            assert sess.compute([y]) == 0, sess.last_error()
            z = plain + (bias if b is not None else 0.0)
            g, u = np.minimum(z[:, ::2], limit), np.clip(z[:, 1::2], -limit, limit)
            want = g * P.sigmoid(alpha * g) * (u + 1.0)
            assert np.allclose(get(sess, y), want, rtol=2 ** -8 if yt == gp.BF16 else 1e-4, atol=2e-4 * max(1.0, np.sqrt(k) / 8))


@TYPES
@pytest.mark.parametrize("n,k,m", [(50, 24, 1), (33, 40, 5), (70, 64, 16), (96, 72, 40), (300, 128, 200), (20, 7, 30)])
def test_a_part_of_the_columns_a_bias_and_an_addend(sess, n, k, m, wt, xt, yt):
    """the two halves of a matrix's columns as weights of their own, the second's result on top of the first's"""
    rng = np.random.default_rng(n + k)
    w, x, x0, bias = M.bf16(rng.standard_normal((n, 2 * k))), M.bf16(rng.standard_normal((m, k))), M.bf16(rng.standard_normal((m, k))), rng.standard_normal(n).astype(np.float32)
    tw = put(sess, w, wt)
    left, right = (strided(sess, tw, k, n, tw.nb[1], h * k * tw.nb[0]) for h in (0, 1))
    z0 = node(sess, DENSE_MM, gp.F32, [n, m], [right, put(sess, x0, xt)])
    y = node(sess, DENSE_MM, yt, [n, m], [left, put(sess, x, xt), z0, None, put(sess, bias)])
    assert sess.compute([z0, y]) == 0, sess.last_error()
    want = np.concatenate([x, x0], axis=1).astype(np.float64) @ w.T.astype(np.float64) + bias
    assert np.allclose(get(sess, y), want, rtol=2 ** -8 if yt == gp.BF16 else 1e-5, atol=1e-4 * np.sqrt(k))


@pytest.mark.parametrize("yt", [gp.F32, gp.BF16])
@pytest.mark.parametrize("k,m", [(1, 2), (37, 3), (48, 1), (512, 40), (4096, 16), (4096, 17), (8192, 20), (9000, 2)])
def test_layer_norms_around_a_sum(sess, k, m, yt):
    rng = np.random.default_rng(k + m)
    x, y = rng.standard_normal((m, k)).astype(np.float32), (3.0 + 50.0 * rng.standard_normal((m, 1)) + rng.standard_normal((m, k))).astype(np.float32)   # far from zero means
    w1, b1, sc, w2, b2 = (rng.standard_normal(k).astype(np.float32) for _ in range(5))
    tx, ty, tw1, tb1, tsc, tw2, tb2 = (put(sess, v) for v in (x, y, w1, b1, sc, w2, b2))
    eps, f = 1e-2, np.float64
    rtol, atol = (2 ** -8, 1e-3) if yt == gp.BF16 else (2e-5, 2e-4)
    for bias, scale, second in ((b1, sc, "norm"), (None, None, "norm"), (b1, None, "same"), (b1, sc, None)):
        h = put(sess, np.zeros((m, k)), yt)
        t = node(sess, NORM_SUM, gp.F32, [k, m], [tx, ty, tw1, tb1 if bias is not None else None, tsc if scale is not None else None,
                                                 tw2 if second == "norm" else None, tb2 if second == "norm" else None, h if second else None], floats=[(0, eps)])
        assert sess.compute([t]) == 0, sess.last_error()
        total = x + L.layer_norm(y.astype(f), w1.astype(f), f(0) if bias is None else bias.astype(f), eps) * (1.0 if scale is None else scale.astype(f))
        assert np.allclose(get(sess, t), total, rtol=2e-5, atol=2e-4)
        after = L.layer_norm(total, w2.astype(f), b2.astype(f), eps) if second == "norm" else total if second else np.zeros((m, k))
        assert np.allclose(get(sess, h), after, rtol=rtol, atol=atol * (10 if k == 1 else 1))
    for bias in (b2, None):
        t = node(sess, LAYER_NORM_W, yt, [k, m], [ty, tw2, tb2 if bias is not None else None], floats=[(0, eps)])
        assert sess.compute([t]) == 0, sess.last_error()
        assert np.allclose(get(sess, t), L.layer_norm(y.astype(f), w2.astype(f), f(0) if bias is None else bias.astype(f), eps), rtol=rtol, atol=atol)


@pytest.mark.parametrize("ty", [gp.F32, gp.BF16])
def test_embeddings_of_token_pairs(sess, ty):
    rng = np.random.default_rng(3)
    k, vocab, spec = 40, 70, {"buckets": 11, "mul_prev": 8, "mul_cur": 10}
    w = {"embed": M.bf16(rng.standard_normal((vocab, k))), "bigram": M.bf16(rng.standard_normal((12, k)))}
    toks = rng.integers(0, vocab, 30)
    prev = np.concatenate([[-1], toks[:-1]])
    prev[13] = -1
    te, tb, tt, tp = put(sess, w["embed"], ty), put(sess, w["bigram"], ty), put(sess, toks, gp.I32), put(sess, prev, gp.I32)
    for pairs in (True, False):
        copy = put(sess, np.zeros((30, k)), gp.BF16)
        y = node(sess, PAIR_EMBED, gp.F32, [k, 30], [te, tt, tp if pairs else None, tb if pairs else None, copy], ints=[(1, 8), (2, 10)], floats=[(0, 2.5)])
        assert sess.compute([y]) == 0, sess.last_error()
        full = {"scale": 2.5, "bigram": spec if pairs else None}
        want = np.concatenate([L.embedding(toks[:13], None, w, full), L.embedding(toks[13:], None, w, full)])
        assert np.allclose(get(sess, y), want, atol=1e-6) and np.allclose(get(sess, copy), want, rtol=2 ** -8)
    bad = node(sess, PAIR_EMBED, gp.F32, [k, 2], [te, put(sess, np.array([1, vocab]), gp.I32)], floats=[(0, 1.0)])
    assert sess.compute([bad]) == 0 and b200.load().kernel_error() == 1 and np.allclose(get(sess, bad)[0], w["embed"][1])


def pad8(x):
    return (x + 7) // 8 * 8


@pytest.mark.parametrize("ct", [gp.F32, gp.BF16])
@pytest.mark.parametrize("H,G,d,e,window,keep,splits", [(2, 1, 16, 16, 9, 3, 1), (6, 2, 20, 12, 70, 5, 4), (9, 1, 40, 24, 33, 0, 8), (4, 4, 8, 72, 0, 0, 2)])
def test_grouped_attention_over_segments(sess, H, G, d, e, window, keep, splits, ct):
    """sequences in scattered cells, both forms of the node, prompts and rows that continue; cells no sequence has stay untouched"""
    rng = np.random.default_rng(H + d)
    rows, past = [5, 1, 8, 3], [90, 0, 33, 2]
    n, per, n_cells = sum(rows), pad8(d) + pad8(e), 300
    rot = {"base": 1000.0, "dims": 8}
    proj = M.bf16(rng.standard_normal((n, (H + G) * d + G * e)))
    sink = rng.standard_normal(H).astype(np.float32)
    cells_free = rng.permutation(n_cells)
    cache = np.zeros((n_cells, G, per), np.float32)
    rnd = M.bf16 if ct == gp.BF16 else (lambda x: x)
    seg, tab, pos, cells, row_seg, want, row0, used = [], [], [], [], [], [], 0, 0
    stored = {}
    for i, (r, p0) in enumerate(zip(rows, past)):
        mine = cells_free[used:used + p0 + r]
        used += p0 + r
        k, v = M.bf16(rng.standard_normal((p0, G, d))), M.bf16(rng.standard_normal((p0, G, e)))
        cache[mine[:p0], :, :d] = k
        cache[mine[:p0], :, pad8(d):pad8(d) + e] = v
        x = proj[row0:row0 + r].astype(np.float64)
        q = np.stack([L.rotate_halves(x[t, :H * d].reshape(H, d), p0 + t, rot) for t in range(r)])
        kn = rnd(np.stack([L.rotate_halves(x[t, H * d:(H + G) * d].reshape(G, d), p0 + t, rot) for t in range(r)]))
        vn = x[:, (H + G) * d:].reshape(r, G, e)
        if ct == gp.BF16:
            q_attn = rnd(q)
        mask = {"size": window, "keep_first": keep} if window else None
        kk, vv = np.concatenate([k, kn]), np.concatenate([v, vn])
        want.append([L.attention(z, kk, vv, sink, 0.3, mask, p0) for z in ((q, q_attn) if ct == gp.BF16 else (q, q))])
        key0 = max(keep, p0 - window + 1) if window else 0
        kept = min(keep, p0 + r) if window else 0
        seg.append([row0, r, 0, 0, p0, len(tab), key0, kept])
        tab += list(mine[:kept]) + list(mine[key0:])
        pos += range(p0, p0 + r)
        cells += list(mine[p0:])
        stored.update({mine[p0 + t]: (kn[t], vn[t]) for t in range(r)})
        row_seg += [i] * r
        row0 += r
    ints = [(0, H), (1, G), (2, d), (3, e), (4, window), (5, keep), (7, 8), (13, splits)]
    floats = [(6, 0.3), (8, 1000.0)]
    tpos, tcells, tail = put(sess, np.array(pos), gp.I32), put(sess, np.array(cells), gp.I32), [put(sess, np.array(z), gp.I32) for z in (row_seg, seg, tab)]
    tproj, tsink = put(sess, proj), put(sess, sink)
    want = [np.concatenate([z[form].reshape(len(z[form]), H * e) for z in want]) for form in (0, 1)]
    for form, code in enumerate((GROUPED_DECODE, GROUPED_ATTN)):
        tc = put(sess, cache.reshape(n_cells, -1), ct)
        y = node(sess, code, gp.F32, [H * e, n], [tproj, tpos, tcells, tc] + tail + [tsink], ints=ints, floats=floats)
        nodes = [y]
        if code == GROUPED_ATTN:
            st = strided(sess, tc, tc.ne[0], n_cells, tc.nb[1])
            st.op = GROUPED_STORE
            for i, z in enumerate((tproj, tpos, tcells)):
                st.src[i] = C.pointer(z)
            for i, z in ints:
                st.op_params[i] = z
            for i, z in floats:
                st.op_params[i] = int(np.float32(z).view(np.int32))
            nodes = [st, y]
        assert sess.compute(nodes) == 0, sess.last_error()
        assert b200.load().kernel_error() == 0
        assert np.abs(get(sess, y) - want[form]).max() < 2e-5 * (1 if ct == gp.F32 else 5)
        after = get(sess, tc).reshape(n_cells, G, per)
        for c in range(n_cells):
            if c in stored:
                tol = 2 ** -7 if ct == gp.BF16 else 1e-5
                assert np.allclose(after[c, :, :d], stored[c][0], atol=tol, rtol=tol) and np.allclose(after[c, :, pad8(d):pad8(d) + e], stored[c][1], atol=1e-6)
                assert not after[c, :, d:pad8(d)].any() and not after[c, :, pad8(d) + e:].any()
            else:
                assert np.array_equal(after[c], rnd(cache[c])), "a cell nobody writes"


def test_lists_that_lack_a_position_are_reported(sess):
    """a segment outside the step, a cell the cache has not, a list that is too short: reported, the other sequence unharmed"""
    H, G, d, n = 2, 1, 8, 24
    rng = np.random.default_rng(2)
    proj = rng.standard_normal((n, (H + 2 * G) * d)).astype(np.float32)
    pos, good = list(range(12)) * 2, [0, 12, 0, 1, 0, 0, 0, 0]
    tab, cells = list(range(24)), list(range(24))
    ints = [(0, H), (1, G), (2, d), (3, d), (4, 6), (13, 2)]
    for code in (GROUPED_DECODE, GROUPED_ATTN):
        results = []
        for bad_seg, bad_tab, bad_cells in ((None, None, None), ([12, 13, 0, 1, 0, 12, 0, 0], None, None), (None, 15, None), ([12, 12, 0, 1, 0, 20, 0, 0], None, None), (None, None, 20)):
            t2, c2 = list(tab), list(cells)
            if bad_tab:
                t2[bad_tab] = 99
            if bad_cells:
                c2[bad_cells] = 99
            seg = [good, bad_seg or [12, 12, 0, 1, 0, 12, 0, 0]]
            cache = put(sess, np.zeros((24, 2 * d)))
            ops = [put(sess, proj), put(sess, np.array(pos), gp.I32), put(sess, np.array(c2), gp.I32), cache]
            y = node(sess, code, gp.F32, [H * d, n], ops + [put(sess, np.array(z), gp.I32) for z in ([0] * 12 + [1] * 12, seg, t2)], ints=ints, floats=[(6, 1.0)])
            assert sess.compute([y]) == 0, sess.last_error()
            err = b200.load().kernel_error()
            results.append(get(sess, y)[:12])
            in_step = code == GROUPED_DECODE and not bad_seg   # (this form takes the step's own positions from proj, and stores their cells)
            expect_clean = bad_seg is None and bad_tab is None and bad_cells is None or (in_step and bad_tab) or (code == GROUPED_ATTN and bad_cells) or (
                code == GROUPED_DECODE and bad_seg and bad_seg[1] == 12)
            assert (err == 0) == bool(expect_clean), (code, bad_seg, bad_tab, bad_cells, err)
            assert np.array_equal(results[0], results[-1])


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
    assert not sess.supports(node(sess, DENSE_MM, gp.F32, [8, 3], [w, x], ints=[(0, 2)]))            # a gate halves the rows
    assert not sess.supports(node(sess, DENSE_MM, gp.F32, [4, 3], [w, x, put(sess, np.zeros((3, 4)))], ints=[(0, 2)]))
    assert not sess.supports(node(sess, DENSE_MM, gp.F32, [8, 3], [w, x, None, None, put(sess, np.zeros(7))]))
    assert not sess.supports(node(sess, NORM_SUM, gp.F32, [16, 3], [x, x, None]))
    assert not sess.supports(node(sess, LAYER_NORM_W, gp.F32, [16, 3], [x, put(sess, np.zeros(16)), put(sess, np.zeros(15))]))
    ids = put(sess, np.zeros(3), gp.I32)
    assert not sess.supports(node(sess, PAIR_EMBED, gp.F32, [16, 3], [x, ids, None, x]))
    for change in ([(0, 3), (1, 2)], [(7, 3)], [(13, 3)], [(13, 16)], [(4, -1)], [(2, 5)]):
        ints = dict([(0, 2), (1, 1), (2, 4), (3, 4), (13, 1)] + change)
        seg = put(sess, np.zeros((1, 8)), gp.I32)
        assert not sess.supports(node(sess, GROUPED_DECODE, gp.F32, [8, 3], [x, ids, ids, put(sess, np.zeros((4, 16))), ids, seg, ids], ints=list(ints.items())))
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
