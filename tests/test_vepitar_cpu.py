"""CPU checks of the restatement of the Vepitar decoders' mechanisms."""
import json

import numpy as np
import pytest

from oracle import layers_ref as R
from stack_util import rel
from vepitar_util import attention, config, dense, general, make_tensors, moe, planted_key_case, planted_state_case

LAYERS = [attention(heads=4, kv_heads=2, dim=8, vdim=6, conv=3, window=7, scale=0.9), general(heads=2, dim=7), attention(heads=3, kv_heads=1, dim=5, vdim=5, conv=2, window=4),
          general(heads=3, dim=5)]


def small(streams=3):
    cfg = config(LAYERS, [moe(6, 2, 12), dense(14), None, moe(4, 3, 9)], width=40, vocab=31, streams=streams)
    return cfg, make_tensors(cfg, 1), np.random.default_rng(0).integers(0, 31, size=30)


def test_restatement_does_not_depend_on_the_cuts():
    cfg, t, tokens = small()
    want, layers = R.forward(cfg, t, tokens)
    assert want.shape == (30, 31) and layers.shape == (4, 30, 40)
    for cuts in ([1] * 30, [2, 28], [7, 1, 22]):
        s, got, i = R.Stepper(cfg, t), [], 0
        for n in cuts:
            got.append(s.step(tokens[i:i + n]))
            i += n
        assert rel(np.concatenate(got), want).max() < 1e-12


def test_decay_stays_within_its_bounds():
    assert np.allclose(R.decay_below_one(np.array([-90.0, 0.0, 90.0])), np.exp([0.0, -0.5 * np.exp(-0.5), -np.exp(-0.5)]))


def test_removal_rule_reads_the_old_state():
    """One head: a stored value is read back, removed at rate a while the next one is stored, and decays per key channel."""
    S = np.zeros((1, 3, 3))
    e = np.eye(3)[:, None]
    one, half = np.ones((1, 1, 3)), np.full((1, 1, 3), 0.5)
    v = np.array([[[1.0, 2.0, 3.0]]])
    assert np.allclose(R.removal_rule(e[:1], 2 * e[:1], v, one, half, e[:1], S), 2 * v)          # nothing to remove yet
    o = R.removal_rule(e[:1], e[:1], 10 * v, one, half, e[:1], S)                                # half of 2 v goes, 10 v comes
    assert np.allclose(o, 11 * v)
    w = np.array([[[0.6, 1.0, 1.0]]])
    R.removal_rule(e[1:2], 0 * e[:1], v, w, 0 * one, e[:1], S)
    assert np.allclose(S[0, 0], 6.6 * v[0, 0]) and not S[0, 1:].any()
    S = np.arange(9.0).reshape(1, 3, 3)
    old, u, a = S[0].copy(), np.array([0.6, 0.0, 0.8]), np.array([0.1, 0.2, 0.3])
    R.removal_rule(e[:1], 0 * e[:1], v, w, a[None, None], u[None, None], S)
    assert np.allclose(S[0], (np.diag(w[0, 0]) - np.outer(a * u, u)) @ old)


def test_sigmoid_weights_are_not_normalized():
    q, k, v = np.zeros((1, 2, 4)), np.ones((6, 1, 4)), np.ones((6, 1, 3))
    o = R.sigmoid_attention(q, k, v, np.array([5]), 1.0, np.array([0.0, np.log(3.0)]), 4)
    assert np.allclose(o[0, 0], 2.0) and np.allclose(o[0, 1], 3.0)
    assert np.allclose(R.sigmoid_attention(q, k[:2], v[:2], np.array([1]), 1.0, np.zeros(2), 4), 1.0)


def test_softmax_choices():
    z = np.log(np.array([0.1, 0.4, 0.2, 0.3]))
    ids, w = R.softmax_route(z + 7.0, 2)
    assert ids.tolist() == [1, 3] and np.allclose(w, [4 / 7, 3 / 7])
    assert R.softmax_route(z, 1)[1].tolist() == [1.0]
    h, P = np.random.default_rng(0).normal(size=(3, 5)), {"up": np.random.default_rng(1).normal(size=(4, 5)), "down": np.eye(4)}
    u = h @ P["up"].T
    assert np.allclose(R.squared_relu_mlp(h, P), np.where(u > 0, u * u, 0))
    assert np.allclose(R.silu_mlp(h, {"gate": P["up"], "up": 2 * P["up"], "down": P["down"]}), 2 * u * u / (1 + np.exp(-u)))


def test_streams_are_mixed_from_the_old_ones():
    x = np.array([[[1.0]], [[10.0]]])
    hc = {"in": np.array([0.5, 2.0]), "out": np.array([3.0, -1.0]), "mix": np.array([[1.0, 4.0], [0.0, 2.0]])}
    assert np.allclose(R.hyper_input(x, hc), 20.5)
    assert np.allclose(R.hyper_update(x, np.array([[7.0]]), hc, 0.5)[:, 0, 0], [1 + 10.5, 4 + 20 - 3.5])


def test_planted_weights_stand_out(tmp_path):
    cfg, t, tokens, _ = planted_key_case(tmp_path / "a", attention(heads=4, kv_heads=2, dim=40, vdim=24, window=30, scale=0.4), 35, 60)
    want = R.Stepper(cfg, t).step(tokens)[-1:]
    other = tokens.copy()
    other[35] = 0
    assert rel(R.Stepper(cfg, t).step(other)[-1:], want)[0] > 0.3
    cfg, t, tokens, _ = planted_state_case(tmp_path / "b", 24, 3, 200)
    want = R.Stepper(cfg, t).step(tokens)[-1:]
    other = tokens.copy()
    other[3] = 0
    assert rel(R.Stepper(cfg, t).step(other)[-1:], want)[0] > 0.3


SPOILS = ["conv", "conv_order", "conv_of_values", "norm_before_conv", "query_norm", "value_norm", "scale", "window", "short_window", "softmax", "pb", "pb_order", "gate", "grouping",
          "decay_sign", "no_decay", "tanh", "w0", "removal_bias", "removal_all", "new_state", "unit_key", "state_order", "head_norm", "general_gate", "general_norm", "receptance",
          "hyper_in", "hyper_out", "mix_transposed", "one_by_one", "mult", "norm_plus", "norm2", "final_plus", "silu", "relu", "not_renormed", "largest_only", "eps", "untied", "state_lost"]


@pytest.mark.parametrize("spoil", SPOILS)
def test_the_test_weights_show_each_mechanism(spoil, monkeypatch):
    """A mistake planted in the restatement changes the logits by hundreds of times the f32 tolerance of the GPU tests."""
    cfg, t, tokens = small()
    if spoil == "eps":
        cfg["norm"]["eps"] = 0.3
    want = R.forward(cfg, t, tokens)[0]
    bad, u = json.loads(json.dumps(cfg)), dict(t)
    L = bad["layers"]

    def put(name, f):
        monkeypatch.setattr(R, name, f)
    conv, rms, att, rule, route, update, linear = R.short_conv, R.rms_norm, R.sigmoid_attention, R.removal_rule, R.softmax_route, R.hyper_update, R.linear
    if spoil == "conv":
        put("short_conv", lambda x, w, *a: (x, conv(x, w, *a)[1]))
    elif spoil == "conv_order":
        put("short_conv", lambda x, w, *a: conv(x, w[:, ::-1], *a))
    elif spoil == "conv_of_values":
        for i in (0, 2):
            u[f"l{i}.mix.v.conv"] = np.eye(L[i]["mixer"]["conv"])[-1] + 0 * t[f"l{i}.mix.v.conv"]
    elif spoil == "norm_before_conv":
        put("short_conv", lambda x, w, *a: conv(rms(x.reshape(len(x), -1, 5 if len(w) % 5 == 0 else 2), 1.0, 1e-5).reshape(x.shape), w, *a))
    elif spoil in ("query_norm", "value_norm"):
        sizes = {(4, 8), (3, 5)} if spoil == "query_norm" else {(2, 6), (1, 5)}
        put("rms_norm", lambda x, w, eps: x if x.ndim == 3 and x.shape[1:] in sizes else rms(x, w, eps))
    elif spoil == "scale":
        L[0]["mixer"]["scale"] *= 1.4
    elif spoil == "window":
        L[0]["mixer"]["mask"]["size"] += 1
    elif spoil == "short_window":
        L[2]["mixer"]["mask"]["size"] -= 1
    elif spoil == "softmax":
        put("sigmoid_attention", lambda q, k, v, pos, scale, bias, window: R.paged_attention(q, k, v, pos, scale, None, window))
    elif spoil == "pb":
        u["l0.mix.pb"] = 0 * t["l0.mix.pb"] - 2
    elif spoil == "pb_order":
        u["l0.mix.pb"] = t["l0.mix.pb"][::-1]
    elif spoil == "gate":
        u["l0.mix.g"] = t["l0.mix.g"][::-1]
    elif spoil == "grouping":
        u["l0.mix.q"] = t["l0.mix.q"].reshape(4, 8, -1)[[0, 2, 1, 3]].reshape(32, -1)
    elif spoil == "decay_sign":
        f = R.decay_below_one
        put("decay_below_one", lambda z: f(-z))
    elif spoil == "no_decay":
        put("decay_below_one", lambda z: 0 * z + 1)
    elif spoil == "tanh":
        for i in (1, 3):
            u[f"l{i}.mix.w2"] = 0 * t[f"l{i}.mix.w2"]
    elif spoil == "w0":
        u["l1.mix.w0"] = t["l1.mix.w0"][::-1]
    elif spoil == "removal_bias":
        u["l1.mix.a.b"] = -t["l1.mix.a.b"]
    elif spoil == "removal_all":
        put("removal_rule", lambda r, k, v, w, a, *s: rule(r, k, v, w, 0 * a + a.mean(axis=2, keepdims=True), *s))
    elif spoil == "new_state":              # removal from the decayed state
        put("removal_rule", lambda r, k, v, w, a, uk, S: np.stack([np.stack([step_decayed(S, h, w[n, h], a[n, h], uk[n, h], k[n, h], v[n, h], r[n, h]) for h in range(r.shape[1])]) for n in range(len(r))]))
    elif spoil == "unit_key":
        put("unit_vectors", lambda x: x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + 1e-6) * 0.5)
    elif spoil == "state_order":
        put("removal_rule", lambda r, k, v, *s: rule(r, v, k, *s))
    elif spoil == "head_norm":
        put("rms_norm", lambda x, w, eps: rms(x.reshape(len(x), 1, -1), 1.0, eps).reshape(x.shape) if x.ndim == 3 and x.shape[1:] in {(2, 7), (3, 5)} else rms(x, w, eps))
    elif spoil == "general_gate":
        u["l1.mix.g"] = 0 * t["l1.mix.g"]
    elif spoil == "general_norm":
        u["l1.mix.norm"] = np.roll(t["l1.mix.norm"], 7)
    elif spoil == "receptance":
        u["l1.mix.r"], u["l1.mix.k"] = t["l1.mix.k"], t["l1.mix.r"]
    elif spoil == "hyper_in":
        for i in range(4):
            u[f"l{i}.hc1.in"] = t[f"l{i}.hc1.in"][::-1]
    elif spoil == "hyper_out":
        u["l1.hc1.out"] = t["l1.hc1.out"][::-1]
    elif spoil == "mix_transposed":
        for k in t:
            if k.endswith("mix") and ".hc" in k:
                u[k] = t[k].T
    elif spoil == "one_by_one":             # later streams from the new ones
        def sequential(x, y, hc, mul):
            x = x.copy()
            for s in range(len(x)):
                x[s] = update(x, y, hc, mul)[s]
            return x
        put("hyper_update", sequential)
    elif spoil == "mult":
        bad["residual_mult"] = 0.5
    elif spoil == "norm_plus":
        u["l1.norm1"] = t["l1.norm1"] - 1
    elif spoil == "norm2":
        u["l1.norm2"] = t["l1.norm1"]
    elif spoil == "final_plus":
        u["final.norm"] = t["final.norm"] - 1
    elif spoil == "silu":
        put("silu", R.gelu_tanh)
        L[0]["mlp"] = L[3]["mlp"] = None
        want = None
    elif spoil == "relu":
        put("squared_relu_mlp", lambda h, P: linear(np.maximum(linear(h, P["up"]), 0), P["down"]))
    elif spoil == "not_renormed":
        put("softmax_route", lambda z, top: (route(z, top)[0], np.exp(z - z.max())[route(z, top)[0]] / np.exp(z - z.max()).sum()))
    elif spoil == "largest_only":
        put("softmax_route", lambda z, top: route(z, 1))
    elif spoil == "untied":
        u["embed"] = t["embed"] * np.linspace(0.5, 1.5, 40)
    elif spoil == "state_lost":
        s = R.Stepper(cfg, t)
        s.step(tokens[:15])
        s.state[1].pop("S")
        assert rel(s.step(tokens[15:]), want[15:]).max() > 0.05
        return
    else:
        bad["norm"]["eps"] = 0.1
    if want is None:
        got = R.forward(bad, u, tokens)[0]
        monkeypatch.undo()
        want = R.forward(bad, u, tokens)[0]
        assert rel(got, want).max() > 0.01
        return
    assert rel(R.forward(bad, u, tokens)[0], want).max() > 0.01


def step_decayed(S, h, w, a, u, k, v, r):
    s = w[:, None] * S[h]
    S[h] = s - np.outer(a * u, u @ s) + np.outer(k, v)
    return S[h].T @ r
