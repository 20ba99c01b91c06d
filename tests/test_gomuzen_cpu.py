"""CPU checks of the restatement of the Gomuzen decoders' mechanisms."""
import json

import numpy as np
import pytest

from gomuzen_util import YARN, config, differential, kept, latent, make_tensors, moe
from oracle import layers_ref as R
from stack_util import rel

LAYERS = [latent(heads=2, dim=6, rot_dim=4, vdim=5, kv_rank=9), differential(heads=4, kv_heads=2, dim=8, vdim=6, dims=6, base=30.0, softcap=5.0, scale=1.5),
          kept(heads=4, kv_heads=2, dim=10, vdim=7, dims=8, base=30.0, window=7, keep=2, softcap=6.0, scale=1.2, scaling=dict(YARN, factor=8.0)),
          kept(heads=3, kv_heads=1, dim=5, vdim=5, dims=2, window=4, keep=1, scaling=None)]


def small():
    cfg = config(LAYERS, [moe(6, 2, 3, 2, 12), moe(8, 3, 2, 1, 10, limit=0.7, scale=2.4), None, moe(4, 1, 2, 1, 9)], width=40, vocab=31, loop=(1, 3, 2))
    return cfg, make_tensors(cfg, 1), np.random.default_rng(0).integers(0, 31, size=30)


def test_restatement_does_not_depend_on_the_cuts():
    cfg, t, tokens = small()
    want, layers = R.forward(cfg, t, tokens)
    assert want.shape == (30, 31) and layers.shape == (6, 30, 40)
    for cuts in ([1] * 30, [2, 28], [7, 1, 22]):
        s, got, i = R.Stepper(cfg, t), [], 0
        for n in cuts:
            got.append(s.step(tokens[i:i + n]))
            i += n
        assert rel(np.concatenate(got), want).max() < 1e-12


def test_order_of_runs():
    c = config([latent()] * 5)
    assert R.layer_runs(c) == [(i, None) for i in range(5)]
    c = config([latent()] * 5, loop=(1, 3, 3))
    assert R.layer_runs(c) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None), (4, None)]
    assert R.layer_runs(config([latent()] * 2, loop=(0, 2, 1))) == [(0, 0), (1, None)]


def test_window_with_kept_first_tokens():
    w = R.windowed_softmax(np.zeros((1, 9)), 8, 3, keep=2)
    assert np.allclose(w, [[0.2, 0.2, 0, 0, 0, 0, 0.2, 0.2, 0.2]])
    assert np.allclose(R.windowed_softmax(np.zeros((1, 4)), 3, 3, keep=2), 0.25)       # they meet
    assert np.allclose(R.windowed_softmax(np.zeros((1, 2)), 1, 3, keep=5), 0.5)


def test_soft_cap():
    assert np.allclose(R.soft_cap(np.array([-1e9, 0.0, 1e-3, 1e9]), 5.0), [-5, 0, 1e-3, 5])


def test_rotation_of_halves():
    rng = np.random.default_rng(2)
    f, mul = R.yarn_frequencies(6, 50.0, {"factor": 2.0, "original": 64, "fast": 8.0, "slow": 1.0})
    q, k = rng.normal(size=(1, 1, 9)), rng.normal(size=(1, 1, 9))
    dot = [(R.rotate_halves(q, np.array([p + 5]), f, mul) * R.rotate_halves(k, np.array([p]), f, mul)).sum() for p in (0, 3, 40)]
    assert np.allclose(dot, dot[0])
    r = R.rotate_halves(q, np.array([4]), f, 1.5)
    assert np.allclose(r[..., 6:], q[..., 6:])
    assert np.isclose(r[0, 0, 1] + 1j * r[0, 0, 4], 1.5 * (q[0, 0, 1] + 1j * q[0, 0, 4]) * np.exp(4j * f[1]))


def test_differential_attention_of_one_token():
    """One token: both maps give its value, so the difference is (1 - lambda) v, normed."""
    m = differential(heads=2, kv_heads=1, dim=4, vdim=6, dims=4, diff=0.25)["mixer"]
    cfg = config([{"type": "attention", "mixer": m}], width=12, vocab=5)
    P = {k[len("l0.mix."):]: v.astype(float) for k, v in make_tensors(cfg, 3).items() if k.startswith("l0.mix.")}
    P["o"] = np.eye(12)
    h = np.random.default_rng(0).normal(size=(1, 12))
    v = P["v"] @ h[0]
    lam = np.exp(P["lq1"] @ P["lk1"]) - np.exp(P["lq2"] @ P["lk2"]) + 0.25
    want = R.rms_norm((1 - lam) * v, 1.0, 1e-5) * 0.75
    assert np.allclose(R.mix_differential(h, P, m, 1e-5, np.array([0]), {}), np.tile(want, 2))


def test_choices_within_groups():
    z = np.array([3.0, -3.0, 1.0, 1.2, 0.5, 0.4])
    s = R.sigmoid(z)
    # group scores: 1.0, 1.5, 1.22; the best expert of all stands in the worst group
    ids, w = R.route(z, np.zeros(6), 3, 1, 2, 2.0)
    assert ids.tolist() == [3, 2] and np.allclose(w, 2 * s[[3, 2]])
    ids, _ = R.route(z, np.zeros(6), 3, 2, 3, 1.0)
    assert ids.tolist() == [3, 2, 4]
    ids, w = R.route(z, np.array([0, 0, -4.0, -4.0, -3.0, -3.1]), 3, 2, 4, 1.0)        # negative choice scores still come before the others
    assert ids.tolist() == [0, 1, 4, 5] and np.allclose(w, s[[0, 1, 4, 5]])
    ids, _ = R.route(z, np.zeros(6), 6, 2, 2, 1.0)                                      # groups of one
    assert ids.tolist() == [0, 3]


def test_experts_are_summed_up():
    cfg, t, _ = small()
    P = {k[len("l0.mlp."):]: v.astype(float) for k, v in t.items() if k.startswith("l0.mlp.")}
    h = np.random.default_rng(1).normal(size=(3, 40))
    out = R.moe_mlp(h, P, cfg["layers"][0]["mlp"])
    for i in range(3):
        ids, w = R.route(P["router"] @ h[i], P["correction"], 3, 2, 2, 1.7)
        want = sum(wi * R.clamped_mlp(h[i:i + 1], {n: P[f"e{e}.{n}"] for n in ("gate", "up", "down")}, 1.5)[0] for e, wi in zip(ids, w))
        assert np.allclose(out[i], want)


SPOILS = ["gate", "gate_order", "latent_norm", "latent_pairs", "latent_scale", "half_pairs", "head_norm", "norm_after_rotation", "map_order", "second_lambda", "diff",
          "diff_factor", "difference_norm", "softcap", "softcap_2", "scale_after_cap", "window", "short_window", "keep", "keep_more", "bias", "value_bias", "grouping",
          "turn_factor", "ramp", "kept_positions", "correction", "corrected_weights", "groups", "group_sum", "masked_to_zero", "renormed", "route_scale", "limit",
          "up_plus_one", "times", "shared_cache", "step", "step_every_layer", "loop_range", "norm2", "eps"]


@pytest.mark.parametrize("spoil", SPOILS)
def test_the_test_weights_show_each_mechanism(spoil, monkeypatch):
    """A mistake planted in the restatement changes the logits by hundreds of times the f32 tolerance of the GPU tests."""
    cfg, t, tokens = small()
    if spoil == "eps":
        cfg["norm"]["eps"] = 0.3
    if spoil == "masked_to_zero":           # choice scores that are all negative
        t["l0.mlp.correction"] = t["l0.mlp.correction"] - 3
    if spoil == "kept_positions":
        tokens = np.random.default_rng(0).integers(0, 31, size=60)
    want = R.forward(cfg, t, tokens)[0]
    bad, u = json.loads(json.dumps(cfg)), dict(t)
    L = bad["layers"]

    def put(name, f):
        monkeypatch.setattr(R, name, f)
    route, halves, pairs, rms, soft, paged = R.route, R.rotate_halves, R.rotate_interleaved, R.rms_norm, R.windowed_softmax, R.paged_attention
    if spoil == "gate":
        del u["l0.mix.g"]
    elif spoil == "gate_order":
        u["l0.mix.g"] = t["l0.mix.g"][::-1]
    elif spoil == "latent_norm":
        u["l0.mix.dkv.norm"] = 0 * t["l0.mix.dkv.norm"] + 1
    elif spoil == "latent_pairs":
        put("rotate_interleaved", lambda x, pos, dims, base: halves(x, pos, R.yarn_frequencies(dims, base)[0], 1.0))
    elif spoil == "latent_scale":
        L[0]["mixer"]["scale"] *= 1.5
    elif spoil == "half_pairs":
        put("rotate_halves", R.rotate_pairs)
    elif spoil == "head_norm":
        put("rms_norm", lambda x, w, eps: rms(x.reshape(x.shape[0], 1, -1), 1.0, eps).reshape(x.shape) * w if x.ndim == 3 and np.ndim(w) else rms(x, w, eps))
    elif spoil == "norm_after_rotation":
        raw = {}

        def late(x, w, eps):
            if x.ndim == 3 and np.ndim(w):
                raw["w"], raw["eps"] = w, eps
                return x
            return rms(x, w, eps)
        put("rms_norm", late)
        put("rotate_halves", lambda x, *a: rms(halves(x, *a), raw.pop("w"), raw["eps"]) if "w" in raw else halves(x, *a))
    elif spoil == "map_order":
        q = t["l1.mix.q"].reshape(4, 2, 8, -1)
        u["l1.mix.q"] = q.transpose(1, 0, 2, 3).reshape(64, -1)
    elif spoil == "second_lambda":
        u["l1.mix.lq2"] = 0 * t["l1.mix.lq2"]
    elif spoil == "diff":
        L[1]["mixer"]["diff"] = 0.6
    elif spoil == "diff_factor":
        u["l1.mix.o"] = t["l1.mix.o"] / (1 - 0.35)
    elif spoil == "difference_norm":
        put("rms_norm", lambda x, w, eps: x if np.ndim(w) == 0 else rms(x, w, eps))
    elif spoil in ("softcap", "softcap_2"):
        L[1 if spoil == "softcap" else 2]["mixer"]["softcap"] = None
    elif spoil == "scale_after_cap":
        put("paged_attention", lambda q, k, v, pos, scale, cap=None, *a, **kw: paged(q, k, v, pos, scale, cap and cap * scale, *a, **kw))
    elif spoil == "window":
        L[2]["mixer"]["mask"]["size"] += 1
    elif spoil == "short_window":
        L[3]["mixer"]["mask"]["size"] -= 1
    elif spoil == "keep":
        L[2]["mixer"]["mask"]["keep_first"] -= 1
    elif spoil == "keep_more":
        L[3]["mixer"]["mask"]["keep_first"] += 1
    elif spoil in ("bias", "value_bias"):
        n = "l2.mix.k.b" if spoil == "bias" else "l2.mix.v.b"
        u[n] = 0 * t[n]
    elif spoil == "grouping":
        u["l2.mix.q"] = t["l2.mix.q"].reshape(4, 10, -1)[[0, 2, 1, 3]].reshape(40, -1)
        u["l2.mix.q.b"] = t["l2.mix.q.b"].reshape(4, 10)[[0, 2, 1, 3]].reshape(-1)
    elif spoil == "turn_factor":
        f = R.yarn_frequencies
        put("yarn_frequencies", lambda *a: (f(*a)[0], 1.0))
    elif spoil == "ramp":
        L[2]["mixer"]["rot"]["scaling"].update(fast=1.5, slow=0.1)
    elif spoil == "kept_positions":         # kept keys turned as if they stood right ahead of the window
        def near(q, k, v, pos, scale, cap=None, window=None, keep=0):
            if not keep:
                return paged(q, k, v, pos, scale, cap, window, keep)
            out = np.zeros((len(q), q.shape[1], v.shape[2]))
            for i, p in enumerate(pos):
                kk = k.copy()
                if p >= window + keep:
                    kk[:keep] = k[p - window - keep + 1:p - window + 1]
                out[i:i + 1] = paged(q[i:i + 1], kk, v, pos[i:i + 1], scale, cap, window, keep)
            return out
        put("paged_attention", near)
    elif spoil == "correction":
        put("route", lambda z, c, *a: route(z, 0 * c, *a))
    elif spoil == "corrected_weights":
        def corrected(z, c, g, k, top, scale):
            ids, _ = route(z, c, g, k, top, scale)
            return ids, (R.sigmoid(z) + c)[ids] * scale
        put("route", corrected)
    elif spoil == "groups":
        put("route", lambda z, c, g, k, *a: route(z, c, 1, 1, *a))
    elif spoil == "group_sum":
        def largest(z, c, g, k, top, scale):
            s, per = R.sigmoid(z), len(z) // g
            order = np.argsort(-(s + c).reshape(g, per).max(axis=1))[:k]
            far = np.where(np.isin(np.arange(len(z)) // per, order), 0, -1e9)
            ids, _ = route(z, c + far, 1, 1, top, scale)
            return ids, s[ids] * scale
        put("route", largest)
    elif spoil == "masked_to_zero":
        def zeroed(z, c, g, k, top, scale):
            s, per = R.sigmoid(z), len(z) // g
            score = [np.sort((s + c)[i * per:(i + 1) * per])[-2:].sum() for i in range(g)]
            choice = np.where(np.isin(np.arange(len(z)) // per, np.argsort(-np.array(score))[:k]), s + c, 0)
            ids = np.argsort(-choice, kind="stable")[:top]
            return ids, s[ids] * scale
        put("route", zeroed)
    elif spoil == "renormed":
        def renormed(*a):
            ids, w = route(*a)
            return ids, w / w.sum() * a[-1]
        put("route", renormed)
    elif spoil == "route_scale":
        L[1]["mlp"]["router"]["scale"] = 1.0
    elif spoil == "limit":
        L[1]["mlp"]["expert"]["limit"] = 1.0
    elif spoil == "up_plus_one":
        put("clamped_mlp", lambda h, P, c: R.linear(np.minimum(R.linear(h, P["gate"]), c) * R.sigmoid(1.702 * np.minimum(R.linear(h, P["gate"]), c))
                                                    * np.clip(R.linear(h, P["up"]), -c, c), P["down"]))
    elif spoil == "times":
        bad["loop"]["times"] = 1
    elif spoil == "shared_cache":
        s = R.Stepper(bad, u)
        s.state[3], s.state[4] = s.state[1], s.state[2]
        got = np.concatenate([s.step([x]) for x in tokens[:4]])
        assert rel(got[1:], want[1:4]).max() > 0.05
        return
    elif spoil == "step":
        u["loop.step"] = t["loop.step"][[0, 0]]
    elif spoil == "step_every_layer":
        f = R.layer_runs
        put("layer_runs", lambda c: [(i, p if p is not None else 0 if i == 2 else None) for i, p in f(c)])
    elif spoil == "loop_range":
        bad["loop"]["stop"] = 2
    elif spoil == "norm2":
        u["l1.norm2"] = t["l1.norm1"]
    else:
        bad["norm"]["eps"] = 0.1
    assert rel(R.forward(bad, u, tokens)[0], want).max() > 0.05
