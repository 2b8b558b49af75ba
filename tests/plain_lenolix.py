"""A plain, slow restatement of the mechanisms of the Lenolix design in numpy float64, one function per mechanism, token by
token where a mechanism has an order.  Test infrastructure like plain_decoder.py (whose softmax, sigmoid and layer order it
uses): it shares no code with the library.  `Plain` strings the mechanisms together for one sequence."""
import math

import numpy as np

from plain_decoder import layer_runs, sigmoid, softmax_with_sink

F = np.float64


def layer_norm(x, w, b, eps):
    mean = x.mean(axis=-1, keepdims=True)
    dev = x - mean
    return dev / np.sqrt((dev * dev).mean(axis=-1, keepdims=True) + eps) * w + b


def pair_row(prev, cur, spec):
    """the row of the table of token pairs; prev None: nothing stands before the token"""
    return spec["buckets"] if prev is None else (int(prev) * spec["mul_prev"] + int(cur) * spec["mul_cur"]) % spec["buckets"]


def embedding(tokens, prev, w, spec):
    """the table's rows times the scale, plus the rows of (token before, token)"""
    out = []
    for t in tokens:
        row = w["embed"][t] * spec["scale"]
        if spec.get("bigram"):
            row = row + w["bigram"][pair_row(prev, t, spec["bigram"])]
        out.append(row)
        prev = t
    return np.array(out)


def frequencies(rot):
    """per pair: base^(-2i/dims); with scaling, long waves are stretched by `factor`, short ones kept, a ramp in between"""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                keep = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = keep * f + (1.0 - keep) * f / sc["factor"]
        out.append(f)
    return np.array(out)


def rotate_halves(x, pos, rot):
    """x [..., d] of one token: channels i and i + dims / 2 are the pairs; channels from dims on pass"""
    half = rot["dims"] // 2
    a = pos * frequencies(rot)
    y = x.copy()
    u, v = x[..., :half], x[..., half:2 * half]
    y[..., :half] = u * np.cos(a) - v * np.sin(a)
    y[..., half:2 * half] = u * np.sin(a) + v * np.cos(a)
    return y


def visible(i, mask):
    """the positions token i sees: a window that ends with itself, and the sequence's first tokens"""
    if not mask:
        return range(i + 1)
    return [j for j in range(i + 1) if j < mask.get("keep_first", 0) or i - j < mask["size"]]


def attention(q, k, v, sink, scale, mask, pos0):
    """q [T, H, d] at positions pos0 .., k [N, G, d], v [N, G, e] of positions 0 .. N - 1 -> [T, H, e]"""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]), F)
    for t in range(T):
        js = visible(pos0 + t, mask)
        if len(js) == js[-1] - js[0] + 1:
            js = slice(js[0], js[-1] + 1)   # (the same positions, without a copy)
        for h in range(H):
            out[t, h] = softmax_with_sink(k[js, h // per] @ q[t, h] * scale, sink[h]) @ v[js, h // per]
    return out


def mixer(h, w, p, mix, past=None, rnd=lambda x: x):
    """h [T, width] -> [T, width], and the keys and values later tokens see"""
    H, G, d, e, T = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"], h.shape[0]
    pos0 = 0 if past is None else past[0].shape[0]
    q, k, v = (h @ w[p + "q"].T).reshape(T, H, d), (h @ w[p + "k"].T).reshape(T, G, d), (h @ w[p + "v"].T).reshape(T, G, e)
    if mix.get("rot"):
        for t in range(T):
            q[t], k[t] = rotate_halves(q[t], pos0 + t, mix["rot"]), rotate_halves(k[t], pos0 + t, mix["rot"])
    q, k, v = rnd(q), rnd(k), rnd(v)
    if past is not None:
        k, v = np.concatenate([past[0], k]), np.concatenate([past[1], v])
    o = attention(q, k, v, w[p + "sink"], mix["scale"], mix.get("mask"), pos0)
    return rnd(o.reshape(T, H * e)) @ w[p + "o"].T, (k, v)


def gated(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, w, p, spec, rnd=lambda x: x):
    return rnd(gated(h @ w[p + "gate"].T, h @ w[p + "up"].T, spec["limit"])) @ w[p + "down"].T


def sublayer(x, f, w, p, which, eps, rnd=lambda x: x):
    """norm, the sublayer, norm, per-channel scale, sum; f returns (rows, what it keeps)"""
    y, kept = f(rnd(layer_norm(x, w[p + "norm" + which], w[p + "norm" + which + ".b"], eps)))
    return x + layer_norm(y, w[p + "norm" + which + "b"], w[p + "norm" + which + "b.b"], eps) * w[p + "ls" + which], kept


def begin_pass(x, x0, w, t, rnd=lambda x: x):
    return rnd(np.concatenate([x, x0], axis=-1)) @ w["loop.in"].T + w["loop.step"][t]


class Plain:
    """One sequence.  feed(tokens) returns the logits of every token fed and keeps what later tokens need; `residuals` has the
    stream after every layer run.  rnd is applied to every row that a reduced-precision implementation may round."""

    def __init__(self, cfg, weights, rnd=lambda x: x):
        self.cfg, self.rnd = cfg, rnd
        self.w = {k: np.asarray(v, dtype=F) for k, v in weights.items()}
        self.kept, self.prev, self.residuals = {}, None, []

    def feed(self, tokens):
        cfg, w, eps, rnd = self.cfg, self.w, self.cfg["norm"]["eps"], self.rnd
        x = x0 = embedding(tokens, self.prev, w, cfg["embedding"])
        self.prev, self.residuals = tokens[-1], []
        for run, (i, t, begins) in enumerate(layer_runs(cfg)):
            lay, p = cfg["layers"][i], f"l{i}."
            if begins:
                x = begin_pass(x, x0, w, t, rnd)
            x, self.kept[run] = sublayer(x, lambda h: mixer(h, w, p + "mix.", lay["mixer"], self.kept.get(run), rnd), w, p, "1", eps, rnd)
            if lay["mlp"]:
                x, _ = sublayer(x, lambda h: (feed_forward(h, w, p + "mlp.", lay["mlp"], rnd), None), w, p, "2", eps, rnd)
            self.residuals.append(x.copy())
        return rnd(layer_norm(x, w["final.norm"], w["final.norm.b"], eps)) @ w["embed"].T
