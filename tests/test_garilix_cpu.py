"""CPU checks of the layer-list decoders' plain restatement and of the host-side helpers."""
import io
import json

import numpy as np
import pytest

from garilix_util import config, delta, latent, make_tensors, mamba
from oracle import layers_ref as R
from stack_util import bf16_round, rel

LAYERS = [delta(heads=2, kv_heads=1, dim=6, vdim=5), latent(heads=2, dim=6, rot_dim=4, vdim=5, kv_rank=8, window=7), mamba(heads=2, vdim=4, state=3),
          latent(heads=1, dim=5, rot_dim=4, vdim=3, kv_rank=8, window=4, kv_from=1)]


def test_restatement_does_not_depend_on_the_cuts():
    cfg = config(LAYERS, width=24, vocab=31, ff=[10, None, 12, 8])
    t = make_tensors(cfg, 1, a_rank=3, g_rank=2)
    tokens = np.random.default_rng(0).integers(0, 31, size=30)
    want, layers = R.forward(cfg, t, tokens)
    assert want.shape == (30, 31) and layers.shape == (4, 30, 24)
    for cuts in ([1] * 30, [2, 28], [7, 1, 22]):
        s = R.Stepper(cfg, t)
        got, i = [], 0
        for n in cuts:
            got.append(s.step(tokens[i:i + n]))
            i += n
        assert rel(np.concatenate(got), want).max() < 1e-12


def test_delta_rule_stores_and_replaces():
    """Orthonormal keys, no decay, full step: reading with a stored key returns its newest value."""
    rng = np.random.default_rng(0)
    k = np.eye(4)[[0, 1, 2, 1]][:, None]
    v = rng.normal(size=(4, 1, 3))
    S = np.zeros((1, 4, 3))
    o = R.delta_rule(k, k, v, np.ones((4, 1)), np.ones((4, 1, 4)), S)
    assert np.allclose(o, v) and np.allclose(S[0, 1], v[3, 0]) and np.allclose(S[0, 0], v[0, 0])
    R.delta_rule(0 * k[:1], k[:1], v[:1], np.zeros((1, 1)), np.array([[[0.5, 1, 1, 0]]]), S)      # decay alone, per key channel
    assert np.allclose(S[0, 0], 0.5 * v[0, 0]) and np.allclose(S[0, 1], v[3, 0]) and not S[0, 3].any()


def test_state_space_scan_is_a_decaying_sum():
    rng = np.random.default_rng(1)
    T, H, N, e = 6, 2, 3, 2
    x, B, C, dt = rng.normal(size=(T, H, e)), rng.normal(size=(T, 1, N)), rng.normal(size=(T, 1, N)), rng.uniform(0.1, 1, size=(T, H))
    A, D = rng.normal(size=H), rng.normal(size=H)
    y = R.ssd_scan(x, B, C, dt, A, D, np.zeros((H, N, e)))
    for t in range(T):
        for h in range(H):
            want = D[h] * x[t, h] + sum(np.exp(-np.exp(A[h]) * dt[j + 1:t + 1, h].sum()) * dt[j, h] * (B[j, 0] @ C[t, 0]) * x[j, h] for j in range(t + 1))
            assert np.allclose(y[t, h], want)


def test_short_convolution_is_causal_with_history():
    rng = np.random.default_rng(2)
    x, w = rng.normal(size=(9, 4)), rng.normal(size=(4, 3))
    y, h = R.short_conv(x, w)
    assert np.allclose(y[0], x[0] * w[:, 2]) and np.allclose(y[5], x[3] * w[:, 0] + x[4] * w[:, 1] + x[5] * w[:, 2])
    a, h = R.short_conv(x[:4], w)
    b, _ = R.short_conv(x[4:], w, None, h)
    assert np.allclose(np.concatenate([a, b]), y)


def test_window_and_rotation():
    w = R.windowed_softmax(np.zeros((1, 8)), 7, 3)
    assert np.allclose(w, [[0] * 5 + [1 / 3] * 3])
    assert np.allclose(R.windowed_softmax(np.zeros((1, 4)), 3, None), 0.25)
    x = np.random.default_rng(3).normal(size=(2, 1, 6))
    r = R.rotate_interleaved(x, np.array([0, 5]), 4, 100.0)
    assert np.allclose(r[0], x[0]) and np.allclose(r[:, :, 4:], x[:, :, 4:])
    z = (x[1, 0, 2] + 1j * x[1, 0, 3]) * np.exp(1j * 5 * 100.0 ** -0.5)
    assert np.allclose([r[1, 0, 2], r[1, 0, 3]], [z.real, z.imag])


@pytest.mark.parametrize("spoil", ["window", "shared", "conv", "decay", "gate", "grouping"])
def test_the_test_weights_show_each_mechanism(spoil):
    """A mistake planted in the restatement changes the logits far beyond the GPU tests' tolerances."""
    cfg = config(LAYERS, width=24, vocab=31, ff=8)
    t = make_tensors(cfg, 1, a_rank=3, g_rank=2)
    tokens = np.random.default_rng(0).integers(0, 31, size=30)
    want = R.forward(cfg, t, tokens)[0]
    bad = json.loads(json.dumps(cfg))
    u = dict(t)
    if spoil == "window":
        bad["layers"][1]["mixer"]["mask"]["size"] += 1
    elif spoil == "shared":
        bad["layers"][3]["mixer"]["mask"]["size"] = 7
    elif spoil == "conv":
        u["l2.mix.conv"] = t["l2.mix.conv"][:, ::-1]
    elif spoil == "decay":
        u["l0.mix.A_log"] = t["l0.mix.A_log"] - 0.5
    elif spoil == "gate":
        u["l0.mix.g2"] = 0 * t["l0.mix.g2"]
    else:
        bad["layers"][2]["mixer"]["norm_groups"] = 1
    assert rel(R.forward(bad, u, tokens)[0], want).max() > 0.2


def test_trace_rows_and_batches():
    from densecore_b200 import trace

    class Fake:
        def __init__(self):
            self.calls, self.free = [], [3, 2, 1, 0]

        def seq_alloc(self):
            return self.free.pop()

        def seq_free(self, s):
            self.free.append(s)

        def forward_batch(self, entries, rows):
            self.calls.append((entries, list(rows)))
            return np.array(rows, np.float32)[:, None] if len(rows) else None
    m = Fake()
    r = trace.Replayer(m)
    lg = r.step([{"id": "x", "tokens": [1, 2, 3], "want": [2, 0, 2]}, {"id": "y", "tokens": [4], "want": []}, {"id": "z", "tokens": [5, 6], "want": [1]}], ["y"])
    assert m.calls[0] == ([(0, [1, 2, 3]), (1, [4]), (2, [5, 6])], [0, 2, 5])
    assert lg[:, 0].tolist() == [2, 0, 2, 5] and sorted(r.seqs) == ["x", "z"]
    assert r.step([{"id": "y", "tokens": [9]}], ["x", "y", "z", "never"]) is None      # the freed slot is taken again
    assert m.calls[1] == ([(1, [9])], []) and sorted(m.free) == [0, 1, 2, 3]
    assert r.step([], []) is None


def test_bf16_rounding_helper():
    import torch
    x = np.random.default_rng(0).normal(size=1000).astype(np.float32)
    assert np.array_equal(bf16_round(x), torch.tensor(x).to(torch.bfloat16).float().numpy())


def test_parts_of_the_library_name_existing_sources():
    import os
    from densecore_b200 import build
    names = {os.path.basename(s)[:-3] for s in build.sources()}
    for part in build.PARTS.values():
        assert set(part) <= names


def test_command_line_parses(monkeypatch):
    from densecore_b200 import __main__ as cli
    a = cli.parser().parse_args(["generate", "--model", "m", "--tokens", "1,2,3", "--max-new", "4"])
    assert a.dtype == "bfloat16" and a.max_new == 4
    monkeypatch.setattr("sys.stdin", io.StringIO("5 6,7\n\n8\n"))
    assert cli.prompts(a) == [[1, 2, 3]]
    a.tokens = None
    assert cli.prompts(a) == [[5, 6, 7], [8]]
