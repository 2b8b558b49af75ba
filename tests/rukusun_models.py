"""Small random models of the Rukusun design for the tests: a configuration and its weights, every weight exactly a BF16 number."""
import numpy as np


def bf16(x):
    """rounded to BF16 (nearest, ties to even), as float32"""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).view(np.float32)


def gla(heads=3, dim=20, vdim=12, tau=4.0, ff=40):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads=3, dim=24, rot=8, rank=40, vdim=16, window=9, scale=None, base=1000.0, ff=40):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "kv_rank": rank, "vdim": vdim, "mask": {"size": window} if window else None,
                      "scale": (dim + rot) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=48, vocab=101, loop=None, eps=3e-6, scale=5.0):
    c = {"architecture": "Rukusun", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed, rank=6, decay=(-2.0, 6.0)):
    """decay: the range of the decay biases (high: slow, far memory; low: strong)"""
    rng = np.random.default_rng(seed)
    E, w = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        w[name] = rng.standard_normal((n, k)) * gain / np.sqrt(k)

    def near(name, n, mean, dev=0.2):
        w[name] = mean + dev * rng.standard_normal(n)

    w["embed"] = rng.standard_normal((cfg["vocab"], E)) / cfg["embedding"]["scale"]
    mat("head", cfg["vocab"], E, 2.0)
    near("final.norm", E, 0.0)
    if cfg.get("loop"):
        w["loop.step"] = 0.7 * rng.standard_normal((cfg["loop"]["times"], E))
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, d, e = m["heads"], m["dim"], m["vdim"]
        near(p + "norm1", E, 0.0)
        if lay["type"] == "gla":
            for n, rows in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e), ("a1", rank)):
                mat(p + "mix." + n, rows, E, 1.5)
            mat(p + "mix.a2", H * d, rank, 1.5)
            w[p + "mix.a2.b"] = rng.uniform(*decay, H * d)
            near(p + "mix.norm", e, 1.0)
        else:
            R, rot = m["kv_rank"], m["rot_dim"]
            mat(p + "mix.q", H * (d + rot), E, 1.5)
            mat(p + "mix.dkv", R + rot, E, 1.5)
            near(p + "mix.dkv.norm", R, 1.0)
            mat(p + "mix.uk", H * d, R, 1.5)
            mat(p + "mix.uv", H * e, R, 1.5)
            w[p + "mix.sink"] = rng.uniform(-1.0, 3.0, H)
            mat(p + "mix.g", H, E, 1.5)
        mat(p + "mix.o", E, H * e, 1.5)
        if lay["mlp"]:
            near(p + "norm2", E, 0.0)
            mat(p + "mlp.up", lay["mlp"]["ff"], E, 1.5)
            mat(p + "mlp.down", E, lay["mlp"]["ff"], 1.5)
    return {k: bf16(v) for k, v in w.items()}


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def error(got, want):
    """per row: root mean square of the difference of the centred logits over that of the wanted ones"""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()
