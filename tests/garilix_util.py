"""Small Garilix decoders with random weights for the tests: configs and tensors."""
from __future__ import annotations

import numpy as np

from stack_util import bf16_round


def delta(heads=3, kv_heads=None, dim=24, vdim=20, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads or heads, "dim": dim, "vdim": vdim, "conv": conv}}


def latent(heads=3, dim=24, rot_dim=8, vdim=20, kv_rank=40, window=21, base=10000.0, kv_from=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale or (dim + rot_dim) ** -0.5,
         "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def mamba(heads=4, vdim=20, state=24, groups=2, norm_groups=2, conv=4):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                                        "conv": conv}}


def config(layers, width=104, vocab=211, ff=88, eps=1e-5):
    """ff: one size for every layer, or a list with None for layers without a feed-forward."""
    out = []
    for i, ly in enumerate(layers):
        f = ff[i] if isinstance(ff, (list, tuple)) else ff
        out.append(dict(ly, mlp={"kind": "dense", "ff": f} if f else None))
    return {"architecture": "Garilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out}


def make_tensors(cfg, seed=0, a_rank=12, g_rank=20):
    """Random bf16-valued tensors whose scales keep every mechanism at work: scores of a few units, decays from
    nearly 1 down to a few percent, step sizes around one half."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    t = {}

    def mat(name, n, k, gain=1.0):
        t[name] = bf16_round(rng.normal(size=(n, k)) * gain / np.sqrt(k))

    def vec(name, n, mean=1.0, dev=0.2):
        t[name] = bf16_round(mean + dev * rng.normal(size=n))
    t["embed"] = bf16_round(rng.normal(size=(V, W)))
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W)
        if ly["type"] == "channel_delta":
            Q, U = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, c in (("q", Q), ("k", Q), ("v", U)):
                mat(p + n, c, W)
                t[p + n + ".conv"] = bf16_round(rng.normal(size=(c, m["conv"])) * 0.6)
            mat(p + "b", m["heads"], W)
            t[p + "A_log"] = bf16_round(rng.uniform(-2.0, 1.0, size=m["heads"]))
            vec(p + "norm", m["vdim"])
            mat(p + "a1", a_rank, W)
            mat(p + "a2", m["heads"] * m["dim"], a_rank)
            vec(p + "dt_bias", m["heads"] * m["dim"], -3.0, 1.5)
            mat(p + "g1", g_rank, W)
            mat(p + "g2", U, g_rank)
            mat(p + "o", W, U)
        elif ly["type"] == "mamba2":
            inner = m["heads"] * m["vdim"]
            C = inner + 2 * m["groups"] * m["state"]
            mat(p + "in", inner + C + m["heads"], W)
            t[p + "conv"] = bf16_round(rng.normal(size=(C, m["conv"])) * 0.6)
            vec(p + "conv.b", C, 0.0)
            vec(p + "dt_bias", m["heads"], -1.0, 1.0)
            t[p + "A_log"] = bf16_round(rng.uniform(-3.0, 1.0, size=m["heads"]))
            vec(p + "D", m["heads"])
            vec(p + "norm", inner)
            mat(p + "o", W, inner)
        else:
            mat(p + "q", m["heads"] * (m["dim"] + m["rot_dim"]), W, 2.0)
            if m.get("kv_from") is None:
                mat(p + "dkv", m["kv_rank"] + m["rot_dim"], W)
                vec(p + "dkv.norm", m["kv_rank"])
            mat(p + "uk", m["heads"] * m["dim"], m["kv_rank"])
            mat(p + "uv", m["heads"] * m["vdim"], m["kv_rank"])
            mat(p + "o", W, m["heads"] * m["vdim"])
        if ly["mlp"]:
            vec(f"l{i}.norm2", W)
            mat(f"l{i}.mlp.gate", ly["mlp"]["ff"], W)
            mat(f"l{i}.mlp.up", ly["mlp"]["ff"], W)
            mat(f"l{i}.mlp.down", W, ly["mlp"]["ff"])
    vec("final.norm", W)
    mat("head", V, W)
    return t
