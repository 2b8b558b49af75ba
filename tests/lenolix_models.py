"""Small random models of the Lenolix design for the tests: a configuration and its weights, every weight exactly a BF16 number."""
import numpy as np

from rukusun_models import bf16, error, tokens  # noqa: F401

RAMP = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}   # with base 500 over 8 dims: one pair kept, one on the ramp, two stretched


def layer(heads=4, kv_heads=2, dim=20, vdim=12, window=9, keep=3, scale=None, rot=8, base=500.0, scaling=RAMP, ff=40, limit=1.5):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                      "mask": {"size": window, "keep_first": keep} if window else None, "rot": {"base": base, "dims": rot, "scaling": scaling and dict(scaling)}},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def config(layers, width=48, vocab=101, loop=None, eps=3e-6, scale=5.0, bigram=(37, 5, 3)):
    c = {"architecture": "Lenolix", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if bigram:
        c["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed):
    rng = np.random.default_rng(seed)
    E, w = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        w[name] = rng.standard_normal((n, k)) * gain / np.sqrt(k)

    def norm(name):
        w[name] = 1.0 + 0.2 * rng.standard_normal(E)
        w[name + ".b"] = 0.3 * rng.standard_normal(E)

    w["embed"] = rng.standard_normal((cfg["vocab"], E)) / cfg["embedding"]["scale"]
    if cfg["embedding"].get("bigram"):
        w["bigram"] = 0.6 * rng.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, E))
    norm("final.norm")
    if cfg.get("loop"):
        mat("loop.in", E, 2 * E, 1.2)
        w["loop.step"] = 0.5 * rng.standard_normal((cfg["loop"]["times"], E))
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        norm(p + "norm1b")
        w[p + "ls1"] = rng.uniform(0.3, 0.9, E)
        for n, rows in (("q", H * d), ("k", G * d), ("v", G * e)):
            mat(p + "mix." + n, rows, E, 1.5)
        w[p + "mix.sink"] = rng.uniform(-1.0, 3.0, H)
        mat(p + "mix.o", E, H * e, 1.5)
        if lay["mlp"]:
            ff = lay["mlp"]["ff"]
            norm(p + "norm2")
            norm(p + "norm2b")
            w[p + "ls2"] = rng.uniform(0.3, 0.9, E)
            mat(p + "mlp.gate", ff, E, 1.5)
            mat(p + "mlp.up", ff, E, 1.5)
            mat(p + "mlp.down", E, ff, 1.5)
    return {k: bf16(v) for k, v in w.items()}


def needle(window, keep, heads=4, kv_heads=2):
    """One attention layer and a token (59) whose key every query wants: seen, its value takes over the output."""
    dim, rot = 16, 4
    cfg = config([layer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=16, window=window, keep=keep, rot=rot, scaling=None, ff=0)], width=48, vocab=60, bigram=None)
    w = weights(cfg, 81)
    ch = cfg["width"] - 1
    w["embed"][:, ch] = 0.0
    w["embed"][:, 0] = 0.6                      # every token asks for it ...
    w["embed"][59, ch] = 2.0                    # ... and it answers on a channel of its own
    for n in ("l0.norm1", "final.norm"):
        w[n], w[n + ".b"] = np.ones(48), np.zeros(48)
    w["l0.mix.k"][:, ch] = 0.0
    for g in range(kv_heads):
        w["l0.mix.k"][g * dim + dim - 1] = 0.0
        w["l0.mix.k"][g * dim + dim - 1, ch] = 4.0
    for h in range(heads):
        w["l0.mix.q"][h * dim + dim - 1] = 0.0
        w["l0.mix.q"][h * dim + dim - 1, 0] = 5.0
    w["l0.mix.v"][:, ch] = 1.0 * np.sign(w["l0.mix.v"][:, 0])
    w["l0.mix.sink"][:] = 1.0
    return cfg, {k: bf16(v) for k, v in w.items()}
