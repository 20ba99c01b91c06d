"""Small Datasun decoders with random weights for the tests: configs and tensors."""
from __future__ import annotations

import numpy as np

from stack_util import bf16_round

YARN = {"factor": 5.0, "original": 96, "fast": 7.0, "slow": 1.5}


def attention(heads=6, kv_heads=2, dim=24, window=21, rot=8, base=900.0, scaling=YARN, scale=None):
    r = {"base": base, "dims": rot}
    if scaling is not None:
        r["scaling"] = dict(scaling)
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window},
                                           "scale": scale or 1.3 * dim ** -0.5, "rot": r}}


def lightning(heads=3, dim=24, vdim=20, decay=None):
    decay = decay or [float(np.exp(-2.0 * 0.5 ** i)) for i in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def config(layers, width=104, vocab=211, ff=88, limit=1.5, eps=1e-5, embed_scale=0.7):
    """ff, limit: one value for every layer, or a list (ff None: no feed-forward)."""
    out = []
    for i, ly in enumerate(layers):
        f = ff[i] if isinstance(ff, (list, tuple)) else ff
        c = limit[i] if isinstance(limit, (list, tuple)) else limit
        out.append(dict(ly, mlp={"kind": "dense", "ff": f, "limit": c} if f else None))
    return {"architecture": "Datasun", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "layers": out}


def make_tensors(cfg, seed=0):
    """Random bf16-valued tensors whose scales keep every mechanism at work: scores of a few units, gate and up values on
    both sides of the limits, biases as large as the projections."""
    rng = np.random.default_rng(seed)
    W, t = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        t[name] = bf16_round(rng.normal(size=(n, k)) * gain / np.sqrt(k))

    def vec(name, n, mean=1.0, dev=0.2):
        t[name] = bf16_round(mean + dev * rng.normal(size=n))
    t["embed"] = bf16_round(rng.normal(size=(cfg["vocab"], W)))
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W)
        if ly["type"] == "attention":
            Q, K = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            mat(p + "q", Q, W)
            mat(p + "k", K, W)
            vec(p + "q.b", Q, 0.0, 0.6)
            vec(p + "k.b", K, 0.3, 0.6)
            vec(p + "q.norm", Q)
            vec(p + "k.norm", K)
            mat(p + "o", W, Q)
            vec(p + "o.b", W, 0.0, 0.5)
        else:
            Q, V = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            mat(p + "q", Q, W)
            mat(p + "k", Q, W)
            mat(p + "v", V, W, 1.5)
            mat(p + "g", V, W)
            vec(p + "norm", V)
            mat(p + "o", W, V, 2.0)
        if ly["mlp"]:
            mat(f"l{i}.mlp.gate", ly["mlp"]["ff"], W, 2.0)
            mat(f"l{i}.mlp.up", ly["mlp"]["ff"], W, 2.0)
            mat(f"l{i}.mlp.down", W, ly["mlp"]["ff"])
    vec("final.norm", W)
    return t
