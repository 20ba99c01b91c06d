"""Datasun decoders through the library against the plain float64 restatement (oracle/layers_ref.py): every mechanism
alone, prompts in portions, mixed batches, reused pages and slots, window edges, long decoding, greedy generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import densecore_b200 as dc
from datasun_util import YARN, attention, config, lightning, make_tensors
from oracle import layers_ref as R
from stack_util import TOL, ModelCase, bf16_round, close, rel, run, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


class Case(ModelCase):
    def __init__(self, path, cfg, n=150, seed=0):
        super().__init__(path, cfg, make_tensors(cfg, seed), n, seed)


STACK = [lightning(heads=4), attention(window=21), lightning(heads=2, dim=40, vdim=12, decay=[0.9995, 0.3]),
         attention(heads=5, kv_heads=5, dim=18, rot=18, window=70, scaling=None), attention(heads=3, kv_heads=1, dim=40, rot=12, window=9),
         lightning(heads=1, dim=16, vdim=72)]


@pytest.fixture(scope="module")
def stack(tmp_path_factory):
    return Case(tmp_path_factory.mktemp("stack"), config(STACK, ff=[88, None, 40, 88, 64, 30], limit=[1.5, 1, 0.7, 3.0, 1.5, 2.5]))


SCALING = dict(YARN)
ALONE = {
    "attention": [attention()],
    "attention_one_head": [attention(heads=1, kv_heads=1, dim=8, rot=2)],
    "attention_many_heads_one_key_head": [attention(heads=9, kv_heads=1, dim=20, rot=6)],
    "attention_every_head_its_own": [attention(heads=3, kv_heads=3, dim=16, rot=16)],
    "attention_odd_sizes": [attention(heads=4, kv_heads=2, dim=17, rot=6, window=13)],
    "attention_96": [attention(heads=6, kv_heads=3, dim=96, rot=32, window=40)],
    "attention_128": [attention(heads=4, kv_heads=1, dim=128, rot=64, window=70)],
    "attention_72": [attention(heads=2, kv_heads=2, dim=72, rot=40, window=33)],
    "attention_200": [attention(heads=2, kv_heads=1, dim=200, rot=100, window=30)],
    "attention_256": [attention(heads=5, kv_heads=1, dim=256, rot=256, window=50)],
    "attention_window_one": [attention(window=1)],
    "attention_window_two": [attention(window=2)],
    "attention_whole_context": [attention(window=5000)],
    "attention_no_scaling": [attention(scaling=None, base=10000.0)],
    "attention_scaling_of_one": [attention(scaling=dict(YARN, factor=1.0))],
    "attention_steep_ramp": [attention(rot=20, base=50.0, scaling=dict(YARN, fast=2.0, slow=1.99))],
    "attention_ramp_below_first_pair": [attention(rot=16, base=400.0, scaling=dict(YARN, original=10, fast=30.0, slow=20.0))],
    "attention_ramp_beyond_last_pair": [attention(rot=6, base=3.0, scaling=dict(YARN, original=100000, fast=2.0, slow=0.01))],
    "attention_strong_scale": [attention(scale=1.0)],
    "attention_windows_and_rotations": [attention(window=5), attention(window=60, base=30.0), attention(window=5, scaling=dict(YARN, factor=2.0))],
    "lightning": [lightning()],
    "lightning_odd_sizes": [lightning(heads=2, dim=17, vdim=5)],
    "lightning_odd_values": [lightning(heads=3, dim=24, vdim=33)],
    "lightning_half_heads": [lightning(heads=3, dim=64, vdim=48)],
    "lightning_full_heads": [lightning(heads=2, dim=128, vdim=128)],
    "lightning_wide_values": [lightning(heads=2, dim=16, vdim=260)],
    "lightning_largest_keys": [lightning(heads=1, dim=256, vdim=96)],
    "lightning_many_heads": [lightning(heads=20, dim=8, vdim=136)],
    "lightning_decays": [lightning(heads=5, decay=[0.0, 1.0, 1e-6, 0.5, 0.99999])],
    "lightning_one_column": [lightning(heads=2, dim=1, vdim=1, decay=[0.7, 0.9])],
}


@pytest.mark.parametrize("name", list(ALONE))
@BOTH
def test_mechanism_alone(ctx, tmp_path, name, dtype):
    """One mixer without a feed-forward: the whole prompt at once, in sixteens, two at a time, and one by one at the end."""
    c = Case(tmp_path, config(ALONE[name], width=72, vocab=131, ff=None), n=140, seed=len(name))
    m = c.model(ctx, dtype)
    for cuts in ([140], [16], [2, 31, 5], [100, 1]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
    m.close()


@pytest.mark.parametrize("limit", [0.05, 1.0, 7.0])
@BOTH
def test_feed_forward_and_odd_widths(ctx, tmp_path, dtype, limit):
    c = Case(tmp_path, config([lightning(heads=1, dim=9, vdim=7), attention(heads=2, kv_heads=1, dim=5, rot=2)], width=50, vocab=77, ff=[37, 300], limit=limit,
                              embed_scale=2.5, eps=1e-2), n=40)
    m = c.model(ctx, dtype)
    assert close(run(m, c.tokens, [40]), c.want, dtype)
    assert close(run(m, c.tokens, [1]), c.want, dtype)
    m.close()


@BOTH
@pytest.mark.parametrize("cuts", [[150], [1], [2], [3, 2, 17], [16, 15], [64, 1, 1, 33], [65, 63], [100, 1]], ids=str)
def test_portions_match_the_whole(ctx, stack, dtype, cuts):
    m = stack.model(ctx, dtype)
    assert close(run(m, stack.tokens, cuts), stack.want, dtype)
    m.close()


@BOTH
def test_steps_larger_than_the_step_buffers(ctx, stack, dtype):
    """Two prompts that together exceed the 32-token step capacity run in several passes of one call."""
    m = stack.model(ctx, dtype, chunk=32)
    a, b = m.seq_alloc(), m.seq_alloc()
    lg = m.forward_batch([(a, stack.tokens[:75]), (b, stack.tokens[:50])], np.arange(125))
    assert close(lg[:75], stack.want[:75], dtype) and close(lg[75:], stack.want[:50], dtype)
    m.close()


@BOTH
def test_mixed_batches_with_reused_pages_and_slots(ctx, stack, dtype):
    """Up to four live requests at different places, portions beside single tokens, ended and started over in a pool
    that holds just them: every logit equals the request's own reference."""
    rng = np.random.default_rng(5)
    m = stack.model(ctx, dtype, max_seqs=4, max_ctx=160, pool_tokens=4 * 160)
    free0 = m.free_blocks()
    live, got, want, seen = {}, [], [], 0
    for step in range(70):
        if len(live) < 4 and rng.random() < 0.5:
            live[m.seq_alloc()] = [0, int(rng.integers(1, 150))]       # position, length
        entries, spans = [], []
        for s, (pos, n) in live.items():
            if rng.random() < 0.2:
                continue
            k = min(int(rng.choice([1, 1, 1, 2, 3, 16, 29, 70])), n - pos)
            entries.append((s, stack.tokens[pos:pos + k]))
            spans.append((s, pos, k))
        if not entries:
            continue
        lg = m.forward_batch(entries, np.arange(sum(k for _, _, k in spans)))
        at = 0
        for s, pos, k in spans:
            got.append(lg[at:at + k])
            want.append(stack.want[pos:pos + k])
            at += k
            live[s][0] += k
            if live[s][0] == live[s][1]:
                m.seq_free(s)
                del live[s]
                seen += 1
    assert seen > 8 and close(np.concatenate(got), np.concatenate(want), dtype)
    for s in live:
        m.seq_free(s)
    assert m.free_blocks() == free0
    m.close()


@BOTH
def test_long_decoding(ctx, tmp_path, dtype):
    """A one-token prompt and 330 decoded tokens: windows and pages pass over decoded keys, states run on."""
    c = Case(tmp_path, config(STACK[:4], ff=48), n=331, seed=9)
    m = c.model(ctx, dtype, max_seqs=1)
    assert close(run(m, c.tokens, [1]), c.want, dtype)
    m.close()


# ---------------------------------------------------------------- keys that stand out
def planted_key_case(path, window, distance, n=None, seed=3):
    """One attention layer whose query of token B finds token A's key far above all others.  A occurs once, B
    `distance` tokens later at the end, so the answer hangs on whether that one key is seen."""
    m = attention(heads=4, kv_heads=2, dim=48, rot=8, window=window, scale=0.36)["mixer"]
    cfg = config([{"type": "attention", "mixer": m}], width=64, vocab=97, ff=None)
    t = make_tensors(cfg, seed)
    A, B, eps = 95, 96, cfg["norm"]["eps"]
    P = {k[len("l0.mix."):]: v.astype(np.float64) for k, v in t.items() if k.startswith("l0.mix.")}
    h = R.rms_norm(t["embed"].astype(np.float64) * cfg["embedding"]["scale"], t["l0.norm1"].astype(np.float64), eps)
    k = R.rms_norm(P["k"] @ h[A] + P["k.b"], P["k.norm"], eps).reshape(2, 48)
    q = P["q"].reshape(4, 48, -1)
    for i in range(4):          # W_q h_B + b = A's key in the dimensions that are not turned
        target = k[i // 2] / P["q.norm"].reshape(4, 48)[i]
        target[:8] = 0
        q[i] += np.outer(target - q[i] @ h[B] - P["q.b"].reshape(4, 48)[i], h[B] / (h[B] @ h[B]))
    t["l0.mix.q"] = bf16_round(q.reshape(192, -1))
    rng = np.random.default_rng(seed)
    tokens = rng.integers(0, 95, size=n or distance + 20)
    tokens[-1], tokens[-1 - distance] = B, A
    return cfg, t, tokens, write_model(path, cfg, t)


@BOTH
@pytest.mark.parametrize("window,distance", [(33, 32), (33, 33), (64, 63), (64, 64), (100, 99), (100, 100), (48, 47), (48, 48), (300, 299), (300, 300),
                                             (129, 128), (129, 129), (300, 16), (300, 17), (2, 1), (2, 2), (1, 1)])
def test_last_key_inside_and_first_outside_the_window(ctx, tmp_path, window, distance, dtype):
    """Seen from a prompt (one step, and a short last portion) and from a decoded token."""
    cfg, t, tokens, path = planted_key_case(tmp_path, window, distance)
    want = R.Stepper(cfg, t).step(tokens)[-1]
    if distance == window or (window > 1 and distance == window - 1):
        cfg["layers"][0]["mixer"]["mask"]["size"] = window + (1 if distance == window else -1)
        assert rel(R.Stepper(cfg, t).step(tokens)[-1][None], want[None])[0] > 0.3       # one token more or less in the window shows
    m = dc.Model.from_dir(ctx, path, dtype, 2, 512)
    m.finalize()
    n = tokens.size
    for cuts in ([n], [n - 1, 1], [n - 2, 2], [n - 18, 18], [max(1, n // 2 - 3), n]):
        assert rel(run(m, tokens, cuts)[-1:], want[None])[0] < TOL[dtype][1], cuts
    m.close()


@BOTH
def test_a_far_key_among_hundreds(ctx, tmp_path, dtype):
    """The standing-out key at every offset of a page, from the first token of the sequence on, decoded and in a portion."""
    for at in list(range(0, 34)) + [255, 256, 399]:
        cfg, t, tokens, path = planted_key_case(tmp_path, 1000, 420 - at, n=421)
        want = R.Stepper(cfg, t).step(tokens)[-1]
        m = dc.Model.from_dir(ctx, path, dtype, 1, 512)
        m.finalize()
        cuts = [[421], [420, 1], [380, 41]][at % 3]
        assert rel(run(m, tokens, cuts)[-1:], want[None])[0] < TOL[dtype][1], at
        m.close()


@BOTH
@pytest.mark.parametrize("bias", [-6.0, 6.0])
def test_sink_share(ctx, tmp_path, bias, dtype):
    """Scores that are all about `bias` times a few: the sink takes nearly everything or nearly nothing, in both kernels."""
    cfg = config([attention(heads=2, kv_heads=1, dim=32, rot=4, window=40, scale=0.25)], width=64, vocab=61, ff=None)
    t = make_tensors(cfg, 4)
    one = np.ones(64, np.float32)
    t["l0.mix.k.b"] = bf16_round(8 * one[:32])                    # keys and queries along one direction
    t["l0.mix.q.b"] = bf16_round(np.sign(bias) * 8 * one)
    cfg["layers"][0]["mixer"]["scale"] = abs(bias) / 32
    path = write_model(tmp_path, cfg, t)
    tokens = np.random.default_rng(1).integers(0, 61, size=90)
    want = R.Stepper(cfg, t).step(tokens)
    f = R.windowed_softmax
    R.windowed_softmax = lambda s, i, w, sink=None: f(s, i, w)
    try:
        without = R.Stepper(cfg, t).step(tokens)
    finally:
        R.windowed_softmax = f
    assert (rel(without, want).max() > 0.3) == (bias < 0)
    m = dc.Model.from_dir(ctx, path, dtype, 1, 128)
    m.finalize()
    for cuts in ([90], [1], [40, 7]):
        assert close(run(m, tokens, cuts), want, dtype), cuts
    m.close()


@BOTH
def test_states_remember(ctx, tmp_path, dtype):
    """Hardly any decay: the first tokens still decide the last logits after 200 more, whatever the cuts, and a slot's
    next sequence starts from nothing."""
    cfg = config([lightning(heads=2, dim=32, vdim=16, decay=[0.9999, 1.0])], width=64, vocab=61, ff=None)
    t = make_tensors(cfg, 2)
    path = write_model(tmp_path, cfg, t)
    tokens = np.random.default_rng(4).integers(0, 61, size=210)
    other = tokens.copy()
    other[:3] = (other[:3] + 1) % 61
    want, want2 = (R.Stepper(cfg, t).step(x)[-1] for x in (tokens, other))
    assert rel(want2[None], want[None])[0] > 5e-3
    m = dc.Model.from_dir(ctx, path, dtype, 1, 512)
    m.finalize()
    for cuts in ([210], [3, 207], [207, 3], [64, 64, 82], [2, 2, 50], [1]):
        for seq, w in ((tokens, want), (other, want2)):
            assert rel(run(m, seq, cuts)[-1:], w[None])[0] < (1e-4 if dtype == "float32" else 2e-2)
    m.close()


@pytest.mark.parametrize("n", [1, 2, 3, 5])
@BOTH
def test_first_tokens(ctx, stack, n, dtype):
    """Short sequences alone and beside a long prompt, on a slot that was used before."""
    m = stack.model(ctx, dtype, max_seqs=2)
    run(m, stack.tokens, [150])
    assert close(run(m, stack.tokens[:n], [n]), stack.want[:n], dtype)
    a, b = m.seq_alloc(), m.seq_alloc()
    lg = m.forward_batch([(a, stack.tokens[:60]), (b, stack.tokens[:n])], np.arange(60 + n))
    assert close(lg[60:], stack.want[:n], dtype)
    m.close()


# ---------------------------------------------------------------- the framework around it
def test_results_do_not_depend_on_the_batch_bitwise(ctx, stack):
    """f32: a request's logits in one ragged batch equal those of the request run alone with the same kernels."""
    m = stack.model(ctx, "float32", max_seqs=3)
    a, b, c = (m.seq_alloc() for _ in range(3))
    lg = m.forward_batch([(a, stack.tokens[:40]), (b, stack.tokens[:90]), (c, stack.tokens[:33])], [39, 129, 162])
    for s in (a, b, c):
        m.seq_free(s)
    alone = []
    for n in (40, 90, 33):
        s = m.seq_alloc()
        alone.append(m.forward_batch([(s, stack.tokens[:n])], [n - 1])[0])
        m.seq_free(s)
    assert np.array_equal(lg, np.stack(alone))
    m.close()


def test_greedy_generation_through_the_scheduler(ctx, stack):
    """Six requests through four slots, prompts in 48-token chunks beside running streams: the reference's tokens."""
    m = stack.model(ctx, "float32", max_seqs=4, max_ctx=192)
    sched = dc.Scheduler(m, max_num_seqs=4, max_prefill_chunk=48)
    prompts = [stack.tokens[i:i + n] for i, n in ((0, 100), (7, 1), (30, 49), (3, 17), (60, 48), (11, 5))]
    ids = [sched.add(p, 12) for p in prompts]
    out = sched.run()
    for i, p in zip(ids, prompts):
        assert out[i] == R.greedy(stack.cfg, stack.tensors, p, 12)
    st = sched.stats()
    assert 1 < st["max_batch"] <= 4 and st["prefill_chunks"] >= 8
    assert st["steps"] < st["prefill_chunks"] + st["decode_steps"]
    sched.close()
    m.close()


@BOTH
def test_entry_points_agree(ctx, stack, dtype):
    """prefill, decode_step, decode_run (device-side feedback), forward_chunk and sampling on one sequence."""
    m = stack.model(ctx, dtype)
    a, b = m.seq_alloc(), m.seq_alloc()
    t0, lg = m.prefill(a, stack.tokens[:90], want_logits=True)
    assert close(lg[None], stack.want[89:90], dtype) and t0 == int(np.argmax(lg))
    assert m.prefill(b, stack.tokens[:90]) == t0
    for _ in range(2):         # eager, captured, replayed
        run_a, ms = m.decode_run([a], [t0], 6)
        step_b, tok = [], t0
        for _ in range(6):
            tok = int(m.decode_step([b], [tok])[0])
            step_b.append(tok)
        assert run_a[:, 0].tolist() == step_b and ms > 0
        t0 = tok
    assert m.seq_len(a) == m.seq_len(b) == 102
    m.seq_free(a)
    m.seq_free(b)
    a = m.seq_alloc()
    assert close(m.forward_chunk(a, stack.tokens[:13]), stack.want[:13], dtype)
    assert close(m.forward_chunk(a, stack.tokens[13:16]), stack.want[13:16], dtype)
    _, lg = m.decode_step([a], [int(stack.tokens[16])], want_logits=True)
    probs = ctx.alloc(4 * m.cfg.vocab)
    tok = dc.spec.sample_dev(m, 0.7, 0.5, probs)
    p = ctx.from_device(probs, np.zeros(m.cfg.vocab, np.float32))
    z = np.exp((lg[0] - lg[0].max()) / 0.7)
    assert np.allclose(p, z / z.sum(), rtol=1e-3, atol=1e-6) and tok == int(np.searchsorted(np.cumsum(p), 0.5))
    ctx.free(probs)
    m.close()


@BOTH
def test_residual_after_every_layer(ctx, stack, dtype):
    _, layers = R.forward(stack.cfg, stack.tensors, stack.tokens[:21])
    m = stack.model(ctx, dtype)
    m.set_option("capture_layer_inputs", 1)
    s = m.seq_alloc()
    for a, b in ((0, 16), (16, 20), (20, 21)):
        m.forward_chunk(s, stack.tokens[a:b])
        for i in range(len(STACK)):
            got = m.read_layer_input(i + 1, b - a)
            assert np.abs(got - layers[i, a:b]).max() < (1e-4 if dtype == "float32" else 0.2) * np.abs(layers[i]).std(), (a, i)
    m.close()


def test_fork_carries_the_state(ctx, stack):
    """A fork shares pages and copies the recurrent state; both continue as if alone."""
    m = stack.model(ctx, "float32")
    a = m.seq_alloc()
    m.forward_batch([(a, stack.tokens[:70])])
    b = m.seq_fork(a)
    other = R.Stepper(stack.cfg, stack.tensors)
    other.step(stack.tokens[:70])
    tail = stack.tokens[100:130]
    want_b = other.step(tail)
    lg = m.forward_batch([(a, stack.tokens[70:100]), (b, tail)], np.arange(60))
    assert close(lg[:30], stack.want[70:100], "float32") and close(lg[30:], want_b, "float32")
    with pytest.raises(dc.DcError, match="recurrent state"):
        m.seq_truncate(a, 10)
    m.close()


def test_without_a_recurrent_layer(ctx, tmp_path):
    """Attention alone: a sequence can be cut back and go on."""
    c = Case(tmp_path, config([attention(), attention(heads=2, window=50)], ff=[None, 30]), n=90)
    m = c.model(ctx, "float32")
    s = m.seq_alloc()
    m.forward_batch([(s, np.concatenate([c.tokens[:50], c.tokens[:20]]))])
    m.seq_truncate(s, 50)
    assert close(m.forward_batch([(s, c.tokens[50:])], np.arange(40)), c.want[50:], "float32")
    m.close()


def test_profile_and_stats(ctx, stack):
    m = stack.model(ctx, "bfloat16")
    s = m.seq_alloc()
    t = m.prefill(s, stack.tokens[:40])
    prof = m.profile_step([s], [t])
    assert {"mixer_in", "mixer_out", "mixer_gqa", "mixer_lightning", "pre_norm", "lm_head_argmax"} <= set(prof)
    launches, wbytes, kvb = m.step_stats()
    assert launches > 20 and 0 < wbytes <= m.weight_bytes() and kvb > 0
    m.close()


def test_random_weights_from_a_config(ctx):
    cfg = config(STACK[:4], ff=48)
    m = dc.Model.from_config(ctx, cfg, max_seqs=1, max_ctx=128)
    m.init_synthetic(5, 0.05)
    m.finalize()
    s = m.seq_alloc()
    _, lg = m.prefill(s, np.arange(50), want_logits=True)
    assert np.isfinite(lg).all() and lg.std() > 0
    m.close()


def test_loading_errors(ctx, tmp_path):
    cfg = config([lightning(), attention()])
    t = make_tensors(cfg)

    def load(name, c=cfg, tensors=t, **kw):
        m = dc.Model.from_dir(ctx, write_model(tmp_path / name, c, tensors, **kw))
        try:
            m.finalize()
        finally:
            m.close()

    def changed(layer, **kw):
        c = json.loads(json.dumps(cfg))
        c["layers"][layer]["mixer"].update(kw)
        return c
    load("good")
    load("f32_vectors", f32=("l0.norm1", "l1.mix.q.b", "final.norm"))
    for name, c, tensors, msg in (
            ("missing", cfg, {k: v for k, v in t.items() if k != "l1.mix.o.b"}, "l1.mix.o.b"),
            ("extra", cfg, dict(t, head=t["embed"]), "head"),
            ("shape", cfg, dict(t, embed=t["embed"][:-1]), "embed"),
            ("mixer", dict(cfg, layers=[dict(cfg["layers"][0], type="mamba2"), cfg["layers"][1]]), t, "mamba2"),
            ("decay", changed(0, decay=[0.5]), t, "decay"),
            ("vdim", changed(1, vdim=12), t, "vdim"),
            ("groups", changed(1, kv_heads=4), t, "kv_heads"),
            ("rotation", changed(1, rot={"base": 100.0, "dims": 26}), t, "dims"),
            ("scaling", changed(1, rot={"base": 100.0, "dims": 8, "scaling": {"factor": 2.0}}), t, "scaling"),
            ("scale", {k: v for k, v in cfg.items() if k != "embedding"}, t, "embedding"),
            ("limit", dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "dense", "ff": 88}), cfg["layers"][1]]), t, "limit")):
        with pytest.raises(dc.DcError, match=msg):
            load(name, c, tensors)


def test_trace_replay_program(ctx, stack, tmp_path):
    """bin/trace_run on interleaved requests: the files hold the wanted logits in the order asked."""
    tk = stack.tokens.tolist()
    steps = [({"step": 0, "entries": [{"id": "a", "tokens": tk[:33], "want": [32, 2]}, {"id": "b", "tokens": tk[:1], "want": [0]}], "end": []}, [32, 2, 0]),
             ({"step": 1, "entries": [{"id": "b", "tokens": tk[1:3], "want": []}], "end": ["b"]}, []),
             ({"step": 2, "entries": [{"id": "c", "tokens": tk[:20], "want": [19]}, {"id": "a", "tokens": tk[33:34], "want": [0]}], "end": ["a", "c"]}, [19, 33])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", stack.path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "130"],
                       input="".join(json.dumps(s) + "\n" for s, _ in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    for s, places in steps:
        f = tmp_path / f"{s['step']}.f32"
        if places:
            assert close(np.fromfile(f, "<f4").reshape(len(places), -1), stack.want[places], "float32")
        else:
            assert not f.exists()


def test_generate_command(stack):
    ps = [stack.tokens[:30].tolist(), stack.tokens[5:9].tolist()]
    r = subprocess.run([sys.executable, "-m", "densecore_b200", "generate", "--model", stack.path, "--dtype", "float32", "--max-new", "6", "--max-ctx", "128"],
                       input="\n".join(",".join(map(str, p)) for p in ps), capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [[int(t) for t in ln.split()] for ln in r.stdout.splitlines()] == [R.greedy(stack.cfg, stack.tensors, p, 6) for p in ps]


@pytest.mark.parametrize("n", [300, 700])
def test_large_products(ctx, tmp_path, n):
    """Enough rows and tokens for the wide tensor-core tiles (more tiles than SMs at the larger size), odd edges included."""
    c = Case(tmp_path, config([lightning(heads=20, dim=24, vdim=40), attention(heads=16, kv_heads=2, dim=48, rot=20, window=200)], width=776, vocab=300,
                              ff=[6500, 3001]), n=n, seed=3)
    m = c.model(ctx, "bfloat16", max_seqs=1, max_ctx=1024)
    assert close(run(m, c.tokens, [n]), c.want, "bfloat16")
    m.close()
