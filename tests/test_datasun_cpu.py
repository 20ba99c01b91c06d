"""CPU checks of the restatement of the Datasun decoders' mechanisms."""
import json

import numpy as np
import pytest

from datasun_util import attention, config, lightning, make_tensors
from oracle import layers_ref as R
from stack_util import rel

LAYERS = [lightning(heads=2, dim=6, vdim=5), attention(heads=4, kv_heads=2, dim=10, rot=8, base=30.0, window=7), lightning(heads=3, dim=4, vdim=3, decay=[0.2, 1.0, 0.97]),
          attention(heads=3, kv_heads=1, dim=5, rot=2, window=4, scaling=None)]


def small():
    cfg = config(LAYERS, width=24, vocab=31, ff=[10, None, 12, 8])
    return cfg, make_tensors(cfg, 1), np.random.default_rng(0).integers(0, 31, size=30)


def test_restatement_does_not_depend_on_the_cuts():
    cfg, t, tokens = small()
    want, layers = R.forward(cfg, t, tokens)
    assert want.shape == (30, 31) and layers.shape == (4, 30, 24)
    for cuts in ([1] * 30, [2, 28], [7, 1, 22]):
        s, got, i = R.Stepper(cfg, t), [], 0
        for n in cuts:
            got.append(s.step(tokens[i:i + n]))
            i += n
        assert rel(np.concatenate(got), want).max() < 1e-12


def test_sink_takes_its_share():
    w = R.windowed_softmax(np.zeros((1, 8)), 7, 3, sink=0.0)
    assert np.allclose(w, [[0] * 5 + [0.25] * 3])
    w = R.windowed_softmax(np.array([[800.0, -800.0]]), 1, 5, sink=0.0)
    assert np.allclose(w, [[1.0, 0.0]])
    assert np.allclose(R.windowed_softmax(np.array([[-900.0]]), 0, 5, sink=0.0), 0.0)


def test_values_are_the_raw_keys():
    """One token: the output is the biased key projection before norm and rotation, less the sink's share."""
    m = attention(heads=2, kv_heads=1, dim=6, rot=4, window=3)["mixer"]
    cfg = config([{"type": "attention", "mixer": m}], width=12, vocab=5, ff=None)
    P = {k[len("l0.mix."):]: v for k, v in make_tensors(cfg, 3).items() if k.startswith("l0.mix.")}
    P["o"], P["o.b"] = np.eye(12), np.zeros(12)
    h = np.random.default_rng(0).normal(size=(1, 12))
    v = P["k"] @ h[0] + P["k.b"]
    k = R.rms_norm(v, P["k.norm"], 1e-5)
    q = R.rms_norm(P["q"] @ h[0] + P["q.b"], P["q.norm"], 1e-5).reshape(2, 6)
    mul = 1 + 0.1 * np.log(5.0)               # at position 0 the turned pairs only grow by the factor
    grow = np.array([mul ** 2] * 4 + [1.0] * 2)
    for i in range(2):
        e = np.exp((q[i] * k * grow).sum() * m["scale"])
        assert np.allclose(R.mix_attention(h, P, m, 1e-5, np.array([0]), {})[0, 6 * i:6 * i + 6], v * e / (1 + e))


def test_linear_attention_is_a_decaying_sum():
    rng = np.random.default_rng(1)
    q, k, v, a = rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 4)), np.array([0.5, 1.0])
    o = R.decayed_linear_attention(q, k, v, a, np.zeros((2, 3, 4)))
    for t in range(6):
        for h in range(2):
            assert np.allclose(o[t, h], sum(a[h] ** (t - i) * (q[t, h] @ k[i, h]) * v[i, h] for i in range(t + 1)))


def test_yarn_ramp():
    f0, one = R.yarn_frequencies(16, 100.0)
    assert one == 1.0 and np.allclose(f0, 100.0 ** (-np.arange(8) / 8))
    f, mul = R.yarn_frequencies(16, 100.0, {"factor": 8.0, "original": 64, "fast": 4.0, "slow": 1.0})
    # pair of t turns: 8 log_100(64 / (2 pi t)): 1.62 for four turns, 4.03 for one; so the ramp runs from pair 1 to pair 5
    ramp = np.clip((np.arange(8) - 1) / 4, 0, 1)
    assert np.allclose(f, f0 * (1 - ramp) + f0 / 8 * ramp) and np.isclose(mul, 1 + 0.1 * np.log(8))
    f, _ = R.yarn_frequencies(8, 100.0, {"factor": 2.0, "original": 4, "fast": 4.0, "slow": 1.0})      # all pairs below the ramp's start of 0
    assert np.allclose(f, R.yarn_frequencies(8, 100.0)[0] * np.where(np.arange(4) > 0, 0.5, 1.0))


def test_rotation_is_relative_and_partial():
    rng = np.random.default_rng(2)
    f, mul = R.yarn_frequencies(6, 50.0)
    q, k = rng.normal(size=(1, 1, 9)), rng.normal(size=(1, 1, 9))
    dot = [(R.rotate_pairs(q, np.array([p + 5]), f, mul) * R.rotate_pairs(k, np.array([p]), f, mul)).sum() for p in (0, 3, 40)]
    assert np.allclose(dot, dot[0])
    r = R.rotate_pairs(q, np.array([4]), f, 1.5)
    assert np.allclose(r[..., 6:], q[..., 6:])
    assert np.isclose(r[0, 0, 2] + 1j * r[0, 0, 3], 1.5 * (q[0, 0, 2] + 1j * q[0, 0, 3]) * np.exp(4j * f[1]))


def test_clamps():
    P = {"gate": np.eye(3), "up": np.eye(3), "down": np.eye(3)}
    x = np.array([[-9.0, 0.4, 9.0]])
    s = R.sigmoid
    assert np.allclose(R.clamped_mlp(x, P, 2.0), [[-9 * s(-9 * 1.702) * (1 - 2), 0.4 * s(0.4 * 1.702) * 1.4, 2 * s(2 * 1.702) * 3]])


SPOILS = ["window", "short_window", "sink", "bias", "head_norm", "grouping", "ramp", "turn_factor", "scale", "decay", "decay_order", "gate",
          "norm_together", "clamp", "clamp_below", "embed_scale", "order", "eps"]


@pytest.mark.parametrize("spoil", SPOILS)
def test_the_test_weights_show_each_mechanism(spoil, monkeypatch):
    """A mistake planted in the restatement changes the logits by hundreds of times the f32 tolerance of the GPU tests."""
    cfg, t, tokens = small()
    if spoil == "eps":
        cfg["norm"]["eps"] = 0.3
    want = R.forward(cfg, t, tokens)[0]
    bad, u = json.loads(json.dumps(cfg)), dict(t)
    L = bad["layers"]
    if spoil == "window":
        L[1]["mixer"]["mask"]["size"] += 1
    elif spoil == "short_window":
        L[3]["mixer"]["mask"]["size"] -= 1
    elif spoil == "sink":
        f = R.windowed_softmax
        monkeypatch.setattr(R, "windowed_softmax", lambda s, i, w, sink=None: f(s, i, w))
    elif spoil == "bias":
        u["l1.mix.k.b"] = 0 * t["l1.mix.k.b"]
    elif spoil == "head_norm":
        f = R.rms_norm

        def per_head(x, w, eps):
            if np.ndim(w) and np.array_equal(w, t["l1.mix.q.norm"]):
                return f(x.reshape(-1, 4, 10), 1.0, eps).reshape(x.shape) * w
            return f(x, w, eps)
        monkeypatch.setattr(R, "rms_norm", per_head)
    elif spoil == "grouping":
        q = t["l1.mix.q"].reshape(4, 10, -1)
        u["l1.mix.q"] = q[[0, 2, 1, 3]].reshape(40, -1)
    elif spoil == "ramp":
        L[1]["mixer"]["rot"]["scaling"]["fast"] = 1.5
        L[1]["mixer"]["rot"]["scaling"]["slow"] = 0.1
    elif spoil == "turn_factor":
        f = R.yarn_frequencies
        monkeypatch.setattr(R, "yarn_frequencies", lambda *a: (f(*a)[0], 1.0))
    elif spoil == "scale":
        L[1]["mixer"]["scale"] *= 1.3
    elif spoil == "decay":
        L[2]["mixer"]["decay"][2] = 0.9
    elif spoil == "decay_order":
        L[0]["mixer"]["decay"].reverse()
    elif spoil == "gate":
        u["l0.mix.g"] = 0 * t["l0.mix.g"]
    elif spoil == "norm_together":
        f = R.rms_norm

        def apart(x, w, eps):
            if np.ndim(w) and np.array_equal(w, t["l2.mix.norm"]):
                return f(x.reshape(-1, 3, 3), 1.0, eps).reshape(x.shape) * w
            return f(x, w, eps)
        monkeypatch.setattr(R, "rms_norm", apart)
    elif spoil == "clamp":
        L[0]["mlp"]["limit"] = 2.0
    elif spoil == "clamp_below":
        monkeypatch.setattr(R, "clamped_mlp", lambda h, P, c: R.linear(
            np.clip(R.linear(h, P["gate"]), -c, c) * R.sigmoid(1.702 * np.clip(R.linear(h, P["gate"]), -c, c)) * (np.clip(R.linear(h, P["up"]), -c, c) + 1), P["down"]))
    elif spoil == "embed_scale":
        bad["embedding"]["scale"] = 1.0
    elif spoil == "order":
        monkeypatch.setattr(R.Stepper, "datasun_layer", _one_after_the_other)
    else:
        bad["norm"]["eps"] = 0.1
    assert rel(R.forward(bad, u, tokens)[0], want).max() > 0.05


def _one_after_the_other(self, i, x, pos, st):
    L, P, eps = self.c["layers"][i], self.part(f"l{i}.mix."), self.c["norm"]["eps"]
    w = self.w[f"l{i}.norm1"]
    h = R.rms_norm(x, w, eps)
    x = x + (R.mix_attention(h, P, L["mixer"], eps, pos, st) if L["type"] == "attention" else R.mix_lightning(h, P, L["mixer"], eps, st))
    if L["mlp"]:
        x = x + R.clamped_mlp(R.rms_norm(x, w, eps), self.part(f"l{i}.mlp."), L["mlp"]["limit"])
    return x
