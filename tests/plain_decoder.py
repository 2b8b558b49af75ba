"""A plain, slow restatement of the mechanisms of decoders with recurrent and latent-attention layers, in numpy float64,
one function per mechanism, token by token.  Test infrastructure: it shares no code with the library and is written from
the equations alone.  `forward` strings the mechanisms together for a model described by a configuration dictionary (the
library's config.json layout) and a dictionary of float arrays under the model's tensor names."""
import numpy as np

F = np.float64


def rms(x, eps):
    """x over its root mean square along the last axis"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm_around_zero(x, w, eps):
    """the weight is stored as its distance from one"""
    return rms(x, eps) * (1.0 + w)


def rms_norm_plain(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rotate_interleaved(x, pos, base, dims):
    """x [..., d] of one token: the pairs (x[2i], x[2i+1]), i < dims / 2, turned by pos * base^(-2i/dims); the rest passes"""
    y = x.copy()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        y[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return y


def window_keys(i, size):
    """the positions token i sees: itself and the size - 1 before it (size None: all before it)"""
    return range(0 if size is None else max(0, i - size + 1), i + 1)


def softmax_with_sink(scores, sink):
    """weights of the keys when exp(sink) stands in the denominator beside them"""
    m = max(scores.max(), sink)
    e = np.exp(scores - m)
    return e / (e.sum() + np.exp(sink - m))


def gla_decay(z, tau):
    """per key channel: sigmoid(z)^(1 / tau)"""
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def gla_recurrence(q, k, v, alpha, state):
    """q, k, alpha [T, H, d], v [T, H, e], state [H, d, e] -> outputs [T, H, e], the state after the last token"""
    S = state.copy()
    out = np.empty(v.shape, F)
    for t in range(q.shape[0]):
        for h in range(q.shape[1]):
            S[h] = alpha[t, h][:, None] * S[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def gla_mixer(h, w, p, mix, eps, state=None, rnd=lambda x: x):
    """h [T, width] -> [T, width] and the state; rnd: see Plain"""
    H, d, e, T = mix["heads"], mix["dim"], mix["vdim"], h.shape[0]
    q = (h @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, e)
    z = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]).reshape(T, H, d)
    if state is None:
        state = np.zeros((H, d, e), F)
    o, state = gla_recurrence(q, k, v, gla_decay(z, mix["tau"]), state)
    o = rms_norm_plain(o, w[p + "norm"], eps).reshape(T, H * e)
    return rnd(o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T, state


def latent_rows(h, w, p, mix, eps, pos0):
    """what a token leaves behind for later ones: its normed latent and its rotated key part"""
    R, rot = mix["kv_rank"], mix["rot_dim"]
    both = h @ w[p + "dkv"].T
    c = rms_norm_plain(both[:, :R], w[p + "dkv.norm"], eps)
    kr = np.stack([rotate_interleaved(both[t, R:R + rot], pos0 + t, mix["rot"]["base"], mix["rot"]["dims"]) for t in range(h.shape[0])])
    return c, kr


def latent_attention(q, c, kr, uk, uv, sink, scale, size, pos0):
    """q [T, H, dim + rot] rotated, at positions pos0 ..; c [N, R], kr [N, rot] of positions 0 .. N - 1; uk [H, dim, R],
    uv [H, vdim, R] -> [T, H, vdim]"""
    T, H, dim = q.shape[0], q.shape[1], uk.shape[1]
    out = np.empty((T, H, uv.shape[1]), F)
    for hd in range(H):
        keys, values = c @ uk[hd].T, c @ uv[hd].T
        for t in range(T):
            js = window_keys(pos0 + t, size)
            lo, hi = js.start, js.stop
            s = (keys[lo:hi] @ q[t, hd, :dim] + kr[lo:hi] @ q[t, hd, dim:]) * scale
            out[t, hd] = softmax_with_sink(s, sink[hd]) @ values[lo:hi]
    return out


def latent_mixer(h, w, p, mix, eps, past=None, rnd=lambda x: x):
    H, dim, rot, R, e, T = mix["heads"], mix["dim"], mix["rot_dim"], mix["kv_rank"], mix["vdim"], h.shape[0]
    pos0 = 0 if past is None else past[0].shape[0]
    q = (h @ w[p + "q"].T).reshape(T, H, dim + rot)
    for t in range(T):
        q[t, :, dim:] = rotate_interleaved(q[t, :, dim:], pos0 + t, mix["rot"]["base"], mix["rot"]["dims"])
    q = rnd(q)
    c, kr = map(rnd, latent_rows(h, w, p, mix, eps, pos0))
    if past is not None:
        c, kr = np.concatenate([past[0], c]), np.concatenate([past[1], kr])
    size = mix["mask"]["size"] if mix.get("mask") else None
    o = latent_attention(q, c, kr, w[p + "uk"].reshape(H, dim, R), w[p + "uv"].reshape(H, e, R), w[p + "sink"], mix["scale"], size, pos0)
    o = rnd(o * sigmoid(h @ w[p + "g"].T)[:, :, None])
    return o.reshape(T, H * e) @ w[p + "o"].T, (c, kr)


def dense_ff(h, w, p, rnd=lambda x: x):
    return rnd(gelu_tanh(h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"gla": gla_mixer, "latent_attention": latent_mixer}


def layer_runs(cfg):
    """[(layer, pass or None, begins a pass)] in the order they run"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    runs = [(i, None, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None, False) for i in range(loop["stop"], n)]


class Plain:
    """One sequence.  feed(tokens) returns the logits of every token fed and keeps what later tokens need.  rnd is applied to every
    row that a reduced-precision implementation may round (what enters a matrix product, queries, cached rows): with it the
    decoder tells how far rounding alone moves the logits."""

    def __init__(self, cfg, weights, rnd=lambda x: x):
        self.cfg, self.rnd = cfg, rnd
        self.w = {k: np.asarray(v, dtype=F) for k, v in weights.items()}
        self.kept = {}
        self.residuals = []

    def feed(self, tokens):
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
        self.residuals = []
        for run, (i, t, begins) in enumerate(layer_runs(cfg)):
            lay, p = cfg["layers"][i], f"l{i}."
            if begins:
                x = x + w["loop.step"][t]
            y, self.kept[run] = MIXERS[lay["type"]](self.rnd(rms_norm_around_zero(x, w[p + "norm1"], eps)), w, p + "mix.", lay["mixer"], eps,
                                                    self.kept.get(run), self.rnd)
            x = x + y
            if lay["mlp"]:
                x = x + dense_ff(self.rnd(rms_norm_around_zero(x, w[p + "norm2"], eps)), w, p + "mlp.", self.rnd)
            self.residuals.append(x.copy())
        return self.rnd(rms_norm_around_zero(x, w["final.norm"], eps)) @ w["head"].T
