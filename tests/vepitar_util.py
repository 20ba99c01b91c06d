"""Small Vepitar decoders with random weights for the tests: configs, tensors, token sequences without close routing calls."""
from __future__ import annotations

import numpy as np

from oracle import layers_ref as R
from stack_util import ModelCase, bf16_round, write_model


def attention(heads=6, kv_heads=2, dim=20, vdim=28, conv=4, window=23, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale or 2.0 * dim ** -0.5}
    return {"type": "attention", "mixer": dict(m, mask={"size": window}) if window else m}


def general(heads=3, dim=24):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}}


def dense(ff=52):
    return {"kind": "dense", "ff": ff}


def moe(experts=10, top=3, ff=36):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, mlp=None, width=104, vocab=211, eps=1e-5, streams=3, mult=0.4):
    """mlp: one feed-forward for every layer, or a list with None for layers without."""
    out = [dict(ly, mlp=mlp[i] if isinstance(mlp, list) else mlp) for i, ly in enumerate(layers)]
    return {"architecture": "Vepitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "residual_mult": mult, "layers": out}


def code_dims(cfg):
    return max([ly["mlp"]["router"]["experts"] for ly in cfg["layers"] if (ly["mlp"] or {}).get("kind") == "moe"], default=0)


def make_tensors(cfg, seed=0, rank=11):
    """Random bf16-valued tensors whose scales keep every mechanism at work.  The last dimensions of the streams hold a code of
    the token that sublayers leave alone and routers read (beside a little of the rest), so that choices have margins that
    rounding does not reach."""
    rng = np.random.default_rng(seed)
    W, V, S, t, n = cfg["width"], cfg["vocab"], cfg["streams"], {}, code_dims(cfg)
    assert n < W

    def mat(name, rows, k, gain=1.0, to_residual=False):
        w = rng.normal(size=(rows, k)) * gain / np.sqrt(k)
        if to_residual and n:
            w[-n:] = 0
        t[name] = bf16_round(w)

    def vec(name, k, mean=0.0, dev=0.2):
        t[name] = bf16_round(mean + dev * rng.normal(size=k))

    def hyper(p):
        vec(p + "in", S, 1.0 / S, 0.6 / S)
        vec(p + "out", S, 1.0, 0.7)
        t[p + "mix"] = bf16_round(0.75 * np.eye(S) + 0.25 / S + 0.2 / S * rng.normal(size=(S, S)))
    embed = rng.normal(size=(V, W))
    for v in range(V):
        embed[v, W - n:] = rng.permutation(np.linspace(-2.0, 2.0, n)) if n > 1 else 1.0
    t["embed"] = bf16_round(embed)
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W)
        if ly["type"] == "attention":
            sizes = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            for k, rows in sizes.items():
                mat(p + k, rows, W)
                w = 0.5 * rng.normal(size=(rows, m["conv"]))
                w[:, -1] += 1.0
                t[p + k + ".conv"] = bf16_round(w)
            vec(p + "pb", m["heads"], -2.0, 0.7)
            mat(p + "g", m["heads"], W, 2.0)
            mat(p + "o", W, m["heads"] * m["vdim"], 0.7, True)
        else:
            Q = m["heads"] * m["dim"]
            for k, gain in (("r", 1.0), ("k", 1.0), ("v", 1.0), ("g", 2.0), ("a", 1.5)):
                mat(p + k, Q, W, gain)
            vec(p + "a.b", Q, 0.0, 0.7)
            mat(p + "w1", rank, W, 1.5)
            mat(p + "w2", Q, rank, 2.0)
            vec(p + "w0", Q, -1.0, 1.0)
            vec(p + "norm", Q, 1.0)
            mat(p + "o", W, Q, 2.0, True)
        hyper(f"l{i}.hc1.")
        if ly["mlp"]:
            p = f"l{i}.mlp."
            vec(f"l{i}.norm2", W, 0.0, 0.1)
            if ly["mlp"]["kind"] == "dense":
                for k in ("gate", "up"):
                    mat(p + k, ly["mlp"]["ff"], W, 1.5)
                mat(p + "down", W, ly["mlp"]["ff"], 1.0, True)
            else:
                e, E = ly["mlp"]["expert"], ly["mlp"]["router"]["experts"]
                w = 0.02 * rng.normal(size=(E, W)) / np.sqrt(W)
                w[:, W - E:] += 1.2 * np.eye(E)[rng.permutation(E)]
                t[p + "router"] = bf16_round(w)
                for x in range(E):
                    mat(f"{p}e{x}.up", e["ff"], W, 1.5)
                    mat(f"{p}e{x}.down", W, e["ff"], 1.0, True)
            hyper(f"l{i}.hc2.")
    vec("final.norm", W)
    return t


def shapes(cfg, rank=11):
    """What a config leaves to the tensors' shapes."""
    return {f"l{i}.mix.w1": [rank, cfg["width"]] for i, ly in enumerate(cfg["layers"]) if ly["type"] == "general_delta"}


def run_with_margins(cfg, tensors, tokens):
    """Logits of every position and the smallest distance of a chosen expert's router logit from the next one."""
    f, per_call = R.softmax_route, []

    def route(z, top):
        order = np.sort(z)[::-1]
        per_call.append(order[top - 1] - order[top] if top < len(z) else np.inf)
        return f(z, top)
    R.softmax_route = route
    try:
        logits = R.Stepper(cfg, tensors).step(tokens)
    finally:
        R.softmax_route = f
    return logits, np.array(per_call).reshape(-1, len(tokens)).min(axis=0) if per_call else np.array([])      # layer by layer, token by token


def settled_tokens(cfg, tensors, tokens, rng, need=0.04):
    """tokens with those replaced whose routing is a close call; and their logits."""
    tokens = np.array(tokens)
    for _ in range(60):
        want, gaps = run_with_margins(cfg, tensors, tokens)
        bad = np.nonzero(gaps < need)[0] if gaps.size else []
        if not len(bad):
            return tokens, want
        for i in bad:
            tokens[i] = rng.integers(0, cfg["vocab"])
    raise AssertionError("no token sequence without close calls")


class Case(ModelCase):
    def __init__(self, path, cfg, n=150, seed=0, tensors=None, rank=11):
        self.cfg, self.tensors = cfg, make_tensors(cfg, seed, rank) if tensors is None else tensors
        self.path = write_model(path, cfg, self.tensors)
        rng = np.random.default_rng(seed + 1)
        self.tokens, self.want = settled_tokens(cfg, self.tensors, rng.integers(0, cfg["vocab"], size=n), rng)


def planted_key_case(path, mixer, at, n, seed=3):
    """One attention layer whose query of token B finds token A's key: that one weight is near 1, the others are small.  A occurs
    once, at place `at`, and B at the end, so the answer hangs on whether that one key is seen."""
    m, W = mixer["mixer"], 64
    cfg = config([mixer], width=W, vocab=97, streams=2)
    t = make_tensors(cfg, seed)
    A, B, H, G, d = 95, 96, m["heads"], m["kv_heads"], m["dim"]
    for k in "qk":                                  # what these heads see of the tokens before is little
        t[f"l0.mix.{k}.conv"][:, :-1] *= 0.03
        t[f"l0.mix.{k}.conv"] = bf16_round(t[f"l0.mix.{k}.conv"])
    u = t["l0.hc1.in"].astype(float).sum() * t["embed"].astype(float)
    h = R.rms_norm(u, 1.0 + t["l0.norm1"].astype(float), cfg["norm"]["eps"])
    own = {k: t[f"l0.mix.{k}.conv"][:, -1].astype(float) for k in "qk"}
    key = (own["k"] * (t["l0.mix.k"].astype(float) @ h[A])).reshape(G, d)
    q = t["l0.mix.q"].astype(float)
    target = key[np.arange(H) // (H // G)].reshape(-1) / own["q"]
    q += np.outer(target - q @ h[B], h[B] / (h[B] @ h[B]))
    t["l0.mix.q"] = bf16_round(q)
    t["l0.mix.pb"] = bf16_round(np.full(H, 6.0 - m["scale"] * d) - 0.1 * np.arange(H))
    t["l0.mix.o"] = bf16_round(20.0 * t["l0.mix.o"])
    tokens = np.random.default_rng(seed).integers(0, 95, size=n)
    tokens[-1], tokens[at] = B, A
    return cfg, t, tokens, write_model(path, cfg, t)


def planted_state_case(path, dim, at, n, seed=5):
    """One recurrent layer that hardly forgets: token A stores a value under a key that token B reads at the end."""
    W = 64
    cfg = config([general(2, dim)], width=W, vocab=97, streams=2)
    t = make_tensors(cfg, seed, rank=5)
    A, B, Q = 95, 96, 2 * dim
    t["l0.mix.w0"] = bf16_round(np.full(Q, -14.0))
    t["l0.mix.w2"] = bf16_round(0.1 * t["l0.mix.w2"])
    t["l0.mix.a.b"] = bf16_round(np.full(Q, -12.0))
    t["embed"][:, :2] = 0                           # A and B are orthogonal to all others
    t["embed"][[A, B]] = 8 * np.eye(W)[:2]
    for k in "kv":                                  # what A stores stands out
        t[f"l0.mix.{k}"] = bf16_round(0.2 * t[f"l0.mix.{k}"])
        t[f"l0.mix.{k}"][:, 0] *= 8
    t["l0.mix.r"][:, 1] = t["l0.mix.k"][:, 0]
    t["l0.mix.o"] = bf16_round(8.0 * t["l0.mix.o"])
    tokens = np.random.default_rng(seed).integers(0, 95, size=n)
    tokens[-1], tokens[at] = B, A
    return cfg, t, tokens, write_model(path, cfg, t)
