"""Small Gomuzen decoders with random weights for the tests: configs, tensors, token sequences without close routing calls."""
from __future__ import annotations

import numpy as np

from oracle import layers_ref as R
from stack_util import ModelCase, bf16_round, write_model

YARN = {"factor": 3.0, "original": 80, "fast": 6.0, "slow": 1.25}


def rot(dims, base, scaling=None):
    r = {"base": base, "dims": dims}
    return dict(r, scaling=dict(scaling)) if scaling else r


def latent(heads=3, dim=20, rot_dim=12, vdim=28, kv_rank=44, base=700.0, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale or 1.2 * (dim + rot_dim) ** -0.5, "rot": rot(rot_dim, base)}}


def differential(heads=4, kv_heads=2, dim=20, vdim=36, dims=12, base=900.0, diff=0.35, softcap=6.0, scale=None, mask=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "softcap": softcap, "scale": scale or 1.5 * dim ** -0.5,
         "rot": rot(dims, base)}
    return {"type": "attention", "mixer": dict(m, mask={"size": mask[0], "keep_first": mask[1]}) if mask else m}


def kept(heads=6, kv_heads=2, dim=24, vdim=20, dims=16, base=300.0, scaling=YARN, softcap=9.0, window=21, keep=3, scale=None):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": softcap, "scale": scale or 1.3 * dim ** -0.5,
                                             "mask": {"size": window, "keep_first": keep}, "rot": rot(dims, base, scaling)}}


def moe(experts=10, top=3, count=2, keep=1, ff=40, limit=1.5, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def config(layers, mlp=None, width=104, vocab=211, eps=1e-5, loop=None):
    """mlp: one feed-forward for every layer, or a list with None for layers without; loop: (start, stop, times)."""
    out = [dict(ly, mlp=mlp[i] if isinstance(mlp, list) else mlp) for i, ly in enumerate(layers)]
    c = {"architecture": "Gomuzen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out}
    return dict(c, loop=dict(zip(("start", "stop", "times"), loop))) if loop else c


def code_dims(cfg):
    return max([ly["mlp"]["router"]["experts"] for ly in cfg["layers"] if ly["mlp"]], default=0)


def make_tensors(cfg, seed=0, correction=0.0):
    """Random bf16-valued tensors whose scales keep every mechanism at work.  The last dimensions of the residual hold a code
    of the token that sublayers leave alone and routers read (beside a little of the rest), so that choices have margins
    that rounding does not reach."""
    rng = np.random.default_rng(seed)
    W, V, t, n = cfg["width"], cfg["vocab"], {}, code_dims(cfg)
    assert n < W

    def mat(name, rows, k, gain=1.0, to_residual=False):
        w = rng.normal(size=(rows, k)) * gain / np.sqrt(k)
        if to_residual and n:
            w[-n:] = 0
        t[name] = bf16_round(w)

    def vec(name, k, mean=1.0, dev=0.2):
        t[name] = bf16_round(mean + dev * rng.normal(size=k))
    embed = rng.normal(size=(V, W))
    for v in range(V):
        embed[v, W - n:] = rng.permutation(np.linspace(-2.0, 2.0, n)) if n > 1 else 1.0
    t["embed"] = bf16_round(embed)
    if cfg.get("loop"):
        t["loop.step"] = bf16_round(0.7 * rng.normal(size=(cfg["loop"]["times"], W)))
        if n:
            t["loop.step"][:, -n:] *= 0.1
        t["loop.step"] = bf16_round(t["loop.step"])
    for i, ly in enumerate(cfg["layers"]):
        m, p, H = ly["mixer"], f"l{i}.mix.", ly["mixer"]["heads"]
        vec(f"l{i}.norm1", W)
        if ly["type"] == "latent_attention":
            mat(p + "q", H * (m["dim"] + m["rot_dim"]), W)
            mat(p + "dkv", m["kv_rank"] + m["rot_dim"], W)
            vec(p + "dkv.norm", m["kv_rank"])
            mat(p + "uk", H * m["dim"], m["kv_rank"])
            mat(p + "uv", H * m["vdim"], m["kv_rank"], 1.5)
            mat(p + "g", H, W, 2.0)
        else:
            maps = 2 if ly["type"] == "attention" else 1
            sizes = {"q": H * maps * m["dim"], "k": m["kv_heads"] * maps * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            for k, rows in sizes.items():
                mat(p + k, rows, W)
                if maps == 1:
                    vec(p + k + ".b", rows, 0.0, 0.6)
            if maps == 2:
                vec(p + "q.norm", m["dim"])
                vec(p + "k.norm", m["dim"])
                for k in ("lq1", "lk1", "lq2", "lk2"):
                    vec(p + k, m["dim"], 0.0, 0.9 * m["dim"] ** -0.25)
        mat(p + "o", W, H * m["vdim"], 1.0, True)
        if ly["mlp"]:
            e, E = ly["mlp"]["expert"], ly["mlp"]["router"]["experts"]
            p = f"l{i}.mlp."
            vec(f"l{i}.norm2", W, 1.0, 0.1)
            w = 0.02 * rng.normal(size=(E, W)) / np.sqrt(W)
            w[:, W - E:] += 1.5 * np.eye(E)[rng.permutation(E)]
            t[p + "router"] = bf16_round(w)
            t[p + "correction"] = bf16_round(correction + 0.15 * rng.normal(size=E))
            for x in range(E):
                mat(f"{p}e{x}.gate", e["ff"], W, 2.0)
                mat(f"{p}e{x}.up", e["ff"], W, 2.0)
                mat(f"{p}e{x}.down", W, e["ff"], 0.4, True)
    vec("final.norm", W)
    mat("head", V, W)
    return t


def margin(z, correction, groups, keep, top):
    """How far the choice scores of a token are from another choice."""
    choice = R.sigmoid(z) + correction
    per, gap = len(z) // groups, np.inf
    score = np.array([np.sort(choice[g * per:(g + 1) * per])[-2:].sum() for g in range(groups)])
    order = np.argsort(-score)
    if keep < groups:
        gap = score[order[keep - 1]] - score[order[keep]]
    rest = np.sort(choice[np.isin(np.arange(len(z)) // per, order[:keep])])[::-1]
    return min(gap, rest[top - 1] - rest[top]) if top < len(rest) else gap


def run_with_margins(cfg, tensors, tokens):
    """Logits of every position and the smallest routing margin of each."""
    gaps, f = [], R.route
    per_call = []

    def route(z, correction, groups, keep, top, scale):
        per_call.append(margin(z, correction, groups, keep, top))
        return f(z, correction, groups, keep, top, scale)
    R.route = route
    try:
        logits = R.Stepper(cfg, tensors).step(tokens)
    finally:
        R.route = f
    if per_call:
        gaps = np.array(per_call).reshape(-1, len(tokens)).min(axis=0)       # layer by layer, token by token
    return logits, np.array(gaps)


def settled_tokens(cfg, tensors, tokens, rng, fixed=(), low=0, high=None, need=0.008):
    """tokens with those replaced (except at the places `fixed`) whose routing is a close call; and their logits."""
    tokens = np.array(tokens)
    for _ in range(60):
        want, gaps = run_with_margins(cfg, tensors, tokens)
        bad = [i for i in np.nonzero(gaps < need)[0] if i not in fixed] if gaps.size else []
        if not bad:
            return tokens, want
        for i in bad:
            tokens[i] = rng.integers(low, high or cfg["vocab"])
    raise AssertionError("no token sequence without close calls")


class Case(ModelCase):
    def __init__(self, path, cfg, n=150, seed=0, tensors=None):
        self.cfg, self.tensors = cfg, make_tensors(cfg, seed) if tensors is None else tensors
        self.path = write_model(path, cfg, self.tensors)
        rng = np.random.default_rng(seed + 1)
        self.tokens, self.want = settled_tokens(cfg, self.tensors, rng.integers(0, cfg["vocab"], size=n), rng)
