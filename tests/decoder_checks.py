"""What the tests of configured models share: expected logits from the plain decoders, feeding a context in portions, model folders."""
import json
import os
import struct

import numpy as np

import plain_decoder
import plain_lenolix
import rukusun_models as M

TOL = 2e-5   # F32 models: of the logits' spread (M.error)
PLAIN = {"Rukusun": plain_decoder.Plain, "Lenolix": plain_lenolix.Plain}


def plain(cfg, w, *rnd):
    """one sequence of the plain decoder of the configuration's architecture"""
    return PLAIN[cfg["architecture"]](cfg, w, *rnd)


class Expected:
    """the plain decoder's logits of a sequence, and per row how far BF16 rounding alone moves them (two ways of rounding: some
    rows of random models are far more sensitive than others)"""

    def __init__(self, cfg, w, toks, dtype="float32"):
        self.rows = plain(cfg, w).feed(toks)
        self.limit = np.full(len(toks), TOL)
        if dtype == "bfloat16":
            shaken = [M.error(plain(cfg, w, lambda x, f=f: M.bf16(x * f) / f).feed(toks), self.rows) for f in (1.0, 1.37)]
            self.limit = 1e-2 + 3.0 * np.maximum(*shaken)

    def __getitem__(self, at):
        part = object.__new__(Expected)
        part.rows, part.limit = self.rows[at], self.limit[at]
        return part


def model(ll, cfg, w, dtype="float32", n_ctx=512, n_batch=512, n_seq=4):
    m = ll.Model(cfg, n_ctx, n_batch, n_seq=n_seq, dtype=dtype)
    m.set_tensors(w)
    return m


def feed(m, toks, sizes, seq=0, at=0):
    """the tokens in portions; logits of every one"""
    out, i = [], 0
    while i < len(toks):
        n = min(next(sizes) if not isinstance(sizes, int) else sizes, len(toks) - i)
        got, _ = m.decode_seqs(toks[i:i + n], np.arange(at + i, at + i + n), [seq] * n, np.arange(n))
        out.append(got)
        i += n
    return np.concatenate(out)


def cycle(*sizes):
    while True:
        yield from sizes


def check(got, want, what=""):
    e = M.error(got, want.rows)
    worst = int((e / want.limit).argmax())
    assert (e < want.limit).all(), f"{what}: row {worst} is {e[worst]:.2e} away ({want.limit[worst]:.2e} allowed)"


def plain_greedy(cfg, w, prompt, n):
    """the plain decoder's continuation, and the smallest lead of a picked token over the next best"""
    p, out = plain(cfg, w), []
    row = p.feed(prompt)[-1]
    gap = np.inf
    for _ in range(n):
        s = np.sort(row)
        gap = min(gap, (s[-1] - s[-2]) / row.std())
        out.append(int(row.argmax()))
        row = p.feed([out[-1]])[-1]
    return out, gap


def write_folder(path, cfg, w):
    table, at, parts = {"__metadata__": {"format": "pt"}}, 0, []
    for k, v in w.items():
        raw = (np.ascontiguousarray(v, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        table[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        parts.append(raw)
    head = json.dumps(table).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(parts))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
