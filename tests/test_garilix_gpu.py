"""Garilix decoders through the library against the plain float64 restatement (oracle/layers_ref.py): every mechanism
alone, prompts in portions, mixed batches, reused pages and slots, window edges, long decoding, greedy generation."""
import numpy as np
import pytest

import densecore_b200 as dc
from garilix_util import config, delta, latent, make_tensors, mamba
from oracle import layers_ref as R
from stack_util import TOL, ModelCase, bf16_round, close, rel, run, write_model

pytestmark = pytest.mark.gpu

STACK = [delta(heads=4, kv_heads=2), latent(window=21), mamba(), latent(window=37, kv_from=1), delta(heads=2, dim=40, vdim=12, conv=3),
         mamba(heads=6, vdim=12, state=12, groups=3, norm_groups=4, conv=2)]


class Case(ModelCase):
    def __init__(self, path, cfg, n=150, seed=0, **kw):
        super().__init__(path, cfg, make_tensors(cfg, seed, **kw), n, seed)


@pytest.fixture(scope="module")
def stack(tmp_path_factory):
    return Case(tmp_path_factory.mktemp("stack"), config(STACK, ff=[88, None, 40, 88, 64, None]))


ALONE = {
    "delta": ([delta()], {}),
    "delta_grouped_heads": ([delta(heads=6, kv_heads=2, dim=32, vdim=36, conv=3)], {}),
    "delta_one_tap_odd_sizes": ([delta(heads=2, dim=17, vdim=5, conv=1)], dict(a_rank=1, g_rank=7)),
    "delta_wide": ([delta(heads=1, dim=136, vdim=130, conv=5)], dict(a_rank=33, g_rank=64)),
    "delta_full_heads": ([delta(heads=2, kv_heads=1, dim=128, vdim=128)], {}),
    "delta_half_heads": ([delta(heads=3, dim=64, vdim=48)], {}),
    "mamba": ([mamba()], {}),
    "mamba_full_state": ([mamba(heads=4, vdim=64, state=128, groups=2, norm_groups=1)], {}),
    "mamba_half_state": ([mamba(heads=3, vdim=40, state=64, groups=1, norm_groups=3, conv=5)], {}),
    "mamba_one_group": ([mamba(heads=3, vdim=17, state=10, groups=1, norm_groups=1, conv=3)], {}),
    "mamba_group_per_head": ([mamba(heads=4, vdim=24, state=130, groups=4, norm_groups=3, conv=1)], {}),
    "latent": ([latent()], {}),
    "latent_window_one": ([latent(window=1)], {}),
    "latent_window_two_odd_rank": ([latent(heads=9, dim=20, rot_dim=6, vdim=33, kv_rank=27, window=2, base=300.0, scale=0.31)], {}),
    "latent_wide": ([latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=264, window=70)], {}),
    "latent_full_rank": ([latent(heads=3, dim=64, rot_dim=32, vdim=64, kv_rank=512, window=40)], {}),
    "latent_largest": ([latent(heads=2, dim=200, rot_dim=64, vdim=200, kv_rank=768, window=60)], {}),
    "latent_whole_context": ([latent(window=4096)], {}),
    "latent_shared_cache": ([latent(window=9), latent(heads=5, dim=16, vdim=40, window=50, kv_from=0), latent(kv_rank=24, rot_dim=4, window=3)], {}),
}


@pytest.mark.parametrize("name", list(ALONE))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mechanism_alone(ctx, tmp_path, name, dtype):
    """One mixer without a feed-forward: the whole prompt at once, in sixteens, and two at a time."""
    layers, kw = ALONE[name]
    c = Case(tmp_path, config(layers, width=72, vocab=131, ff=None), n=90, seed=len(name), **kw)
    m = c.model(ctx, dtype)
    for cuts in ([90], [16], [2, 31, 5]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_feed_forward_and_odd_widths(ctx, tmp_path, dtype):
    c = Case(tmp_path, config([delta(heads=1, dim=8, vdim=8), mamba(heads=2, vdim=6, state=4, groups=1, norm_groups=3)], width=50, vocab=77, ff=[37, 300]), n=40)
    m = c.model(ctx, dtype)
    assert close(run(m, c.tokens, [40]), c.want, dtype)
    assert close(run(m, c.tokens, [1]), c.want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cuts", [[150], [1], [2], [3, 2, 17], [16, 15], [64, 1, 1, 33], [100, 1]], ids=str)
def test_portions_match_the_whole(ctx, stack, dtype, cuts):
    m = stack.model(ctx, dtype)
    assert close(run(m, stack.tokens, cuts), stack.want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_steps_larger_than_the_step_buffers(ctx, stack, dtype):
    """Two prompts that together exceed the 32-token step capacity run in several passes of one call."""
    m = stack.model(ctx, dtype, chunk=32)
    a, b = m.seq_alloc(), m.seq_alloc()
    lg = m.forward_batch([(a, stack.tokens[:75]), (b, stack.tokens[:50])], np.arange(125))
    assert close(lg[:75], stack.want[:75], dtype) and close(lg[75:], stack.want[:50], dtype)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
        total = sum(k for _, _, k in spans)
        lg = m.forward_batch(entries, np.arange(total))
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(ctx, tmp_path, dtype):
    """A one-token prompt and 330 decoded tokens: windows and pages pass over decoded keys, states run on."""
    c = Case(tmp_path, config(STACK[:4], ff=48), n=331, seed=9)
    m = c.model(ctx, dtype, max_seqs=1)
    assert close(run(m, c.tokens, [1]), c.want, dtype)
    m.close()


# ---------------------------------------------------------------- keys that stand out
def planted_key_case(path, window, distance, head_window=None, n=None, seed=3):
    """One attention layer whose query of token B finds token A's key far above all others.  A occurs once, B
    `distance` tokens later at the end, so the answer hangs on whether that one key is seen."""
    cfg = config([latent(heads=2, dim=16, rot_dim=4, vdim=16, kv_rank=32, window=window)], width=64, vocab=97, ff=None)
    t = make_tensors(cfg, seed)
    A, B = 95, 96
    m, x = cfg["layers"][0]["mixer"], t["embed"].astype(np.float64)
    P = {k[len("l0.mix."):]: v.astype(np.float64) for k, v in t.items() if k.startswith("l0.mix.")}
    c = R.rms_norm((x[A] @ P["dkv"].T)[:m["kv_rank"]], P["dkv.norm"], cfg["norm"]["eps"])
    ku = (P["uk"] @ c).reshape(m["heads"], m["dim"])
    q = t["l0.mix.q"].reshape(m["heads"], m["dim"] + m["rot_dim"], -1).copy()
    for h in range(m["heads"]):      # W_q B = a large multiple of A's key (and nothing in the rotated part)
        target = np.zeros(m["dim"] + m["rot_dim"])
        target[:m["dim"]] = ku[h] * (14.0 / m["scale"] / (ku[h] @ ku[h]))
        q[h] += np.outer(target - q[h] @ x[B], x[B] / (x[B] @ x[B])).astype(np.float32)
    t["l0.mix.q"] = bf16_round(q.reshape(t["l0.mix.q"].shape))
    rng = np.random.default_rng(seed)
    tokens = rng.integers(0, 95, size=n or distance + 20)
    tokens[-1], tokens[-1 - distance] = B, A
    return cfg, t, tokens, write_model(path, cfg, t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,distance", [(33, 32), (33, 33), (64, 63), (64, 64), (100, 99), (100, 100), (48, 47), (48, 48), (300, 299), (300, 300),
                                             (300, 16), (300, 17), (2, 1), (2, 2), (1, 1)])
def test_last_key_inside_and_first_outside_the_window(ctx, tmp_path, window, distance, dtype):
    """Seen from a prompt (one step, and a short last portion) and from a decoded token."""
    cfg, t, tokens, path = planted_key_case(tmp_path, window, distance)
    want = R.Stepper(cfg, t).step(tokens)[-1]
    cfg["layers"][0]["mixer"]["mask"]["size"] = window + (1 if distance == window else -1)
    if distance == window or (window > 1 and distance == window - 1):
        wrong = R.Stepper(cfg, t).step(tokens)[-1]
        assert rel(wrong[None], want[None])[0] > 0.3       # one token more or less in the window shows
    m = dc.Model.from_dir(ctx, path, dtype, 2, 512)
    m.finalize()
    n = tokens.size
    for cuts in ([n], [n - 1, 1], [n - 2, 2], [n - 18, 18], [max(1, n // 2 - 3), n]):
        assert rel(run(m, tokens, cuts)[-1:], want[None])[0] < TOL[dtype][1], cuts
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["delta", "mamba"])
def test_states_remember(ctx, tmp_path, kind, dtype):
    """Hardly any decay: the first tokens still decide the last logits after 200 more, whatever the cuts, and a slot's
    next sequence starts from nothing."""
    layer = delta(heads=2, dim=32, vdim=16) if kind == "delta" else mamba(heads=2, vdim=16, state=16, groups=1, norm_groups=2)
    cfg = config([layer], width=64, vocab=61, ff=None)
    t = make_tensors(cfg, 2)
    t["l0.mix.A_log"][:] = -8.0
    if kind == "delta":
        t["l0.mix.b"] *= 0.0625
    path = write_model(tmp_path, cfg, t)
    rng = np.random.default_rng(4)
    tokens = rng.integers(0, 61, size=210)
    other = tokens.copy()
    other[:3] = (other[:3] + 1) % 61
    want, want2 = (R.Stepper(cfg, t).step(x)[-1] for x in (tokens, other))
    assert rel(want2[None], want[None])[0] > 5e-3
    m = dc.Model.from_dir(ctx, path, dtype, 1, 512)
    m.finalize()
    for cuts in ([210], [3, 207], [207, 3], [2, 2, 50], [1]):
        for seq, w in ((tokens, want), (other, want2)):
            assert rel(run(m, seq, cuts)[-1:], w[None])[0] < (1e-4 if dtype == "float32" else 5e-2)
    m.close()


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens(ctx, stack, n, dtype):
    """Sequences shorter than the convolutions, alone and beside a long prompt, on a slot that was used before."""
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
    # one batch holds a prompt chunk and the running streams' tokens: fewer steps than chunks plus decode steps
    assert st["steps"] < st["prefill_chunks"] + st["decode_steps"]
    sched.close()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
    m.close()


def test_what_a_recurrent_state_rules_out(ctx, stack):
    m = stack.model(ctx, "float32", max_seqs=1, max_ctx=64)
    s = m.seq_alloc()
    m.forward_batch([(s, stack.tokens[:20])])
    with pytest.raises(dc.DcError, match="recurrent state"):
        m.seq_truncate(s, 10)
    m.seq_truncate(s, 0)                                     # starting over is fine
    assert close(m.forward_batch([(s, stack.tokens[:30])], np.arange(30)), stack.want[:30], "float32")
    with pytest.raises(dc.DcError, match="does not apply"):
        m.set_option("prefix_cache", 1)
    for entries, rows in (([(s, [0] * 60)], []), ([(s, [10 ** 6])], []), ([(s, [1]), (s, [2])], []), ([(s, [1])], [1]), ([(3, [1])], [])):
        with pytest.raises(dc.DcError):
            m.forward_batch(entries, rows)
    assert m.seq_len(s) == 30
    m.close()


def test_profile_and_stats(ctx, stack):
    m = stack.model(ctx, "bfloat16")
    s = m.seq_alloc()
    t = m.prefill(s, stack.tokens[:40])
    prof = m.profile_step([s], [t])
    assert {"mixer_in", "mixer_out", "mixer_delta", "mixer_ssd", "mixer_latent", "post_norm", "lm_head_argmax"} <= set(prof)
    launches, wbytes, kvb = m.step_stats()
    assert launches > 20 and 0 < wbytes <= m.weight_bytes() and kvb > 0
    m.close()


def test_random_weights_from_a_config(ctx):
    cfg = config(STACK[:4], ff=48)
    shapes = {"l0.mix.a1": [16, 104], "l0.mix.g1": [8, 104]}
    m = dc.Model.from_config(ctx, cfg, shapes, max_seqs=1, max_ctx=128)
    m.init_synthetic(5, 0.05)
    m.finalize()
    s = m.seq_alloc()
    _, lg = m.prefill(s, np.arange(50), want_logits=True)
    assert np.isfinite(lg).all() and lg.std() > 0
    m.close()
    with pytest.raises(dc.DcError, match="shape of tensor"):
        dc.Model.from_config(ctx, cfg, {})


def test_loading_errors(ctx, tmp_path):
    cfg = config([delta(), latent()])
    t = make_tensors(cfg)

    def load(name, c=cfg, tensors=t, **kw):
        m = dc.Model.from_dir(ctx, write_model(tmp_path / name, c, tensors, **kw))
        try:
            m.finalize()
        finally:
            m.close()
    load("good")
    load("f32_vectors", f32=("l0.norm1", "l0.mix.A_log", "final.norm"))
    for name, c, tensors, msg in (
            ("missing", cfg, {k: v for k, v in t.items() if k != "l1.mix.uv"}, "l1.mix.uv"),
            ("extra", cfg, dict(t, unknown=t["head"]), "unknown"),
            ("shape", cfg, dict(t, head=t["head"][:-1]), "head"),
            ("arch", dict(cfg, architecture="Other"), t, "Other"),
            ("mixer", dict(cfg, layers=[dict(cfg["layers"][0], type="other"), cfg["layers"][1]]), t, "other"),
            ("size", dict(cfg, layers=[dict(cfg["layers"][0], mixer={k: v for k, v in cfg["layers"][0]["mixer"].items() if k != "dim"}), cfg["layers"][1]]),
             t, "dim"),
            ("kv_from", config([delta(), latent(kv_from=0)]), t, "kv_from")):
        with pytest.raises(dc.DcError, match=msg):
            load(name, c, tensors)
    with pytest.raises(dc.DcError, match="config.json"):
        dc.Model.from_dir(ctx, str(tmp_path / "nowhere"))
    with open(tmp_path / "good" / "model.safetensors", "r+b") as f:
        f.truncate(4000)
    with pytest.raises(dc.DcError):
        dc.Model.from_dir(ctx, str(tmp_path / "good"))


def test_trace_replay_program(ctx, stack, tmp_path):
    """bin/trace_run on interleaved requests: the files hold the wanted logits in the order asked."""
    import json
    import os
    import subprocess
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    tk = stack.tokens.tolist()
    steps = [({"step": 0, "entries": [{"id": "a", "tokens": tk[:33], "want": [32, 2]}, {"id": "b", "tokens": tk[:1], "want": [0]}], "end": []}, [32, 2, 0]),
             ({"step": 1, "entries": [{"id": "b", "tokens": tk[1:3], "want": []}], "end": ["b"]}, []),
             ({"step": 2, "entries": [{"id": "c", "tokens": tk[:20], "want": [19]}, {"id": "a", "tokens": tk[33:34], "want": [0]}], "end": ["a", "c"]}, [19, 33])]
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", stack.path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "130"],
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
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    ps = [stack.tokens[:30].tolist(), stack.tokens[5:9].tolist()]
    r = subprocess.run([sys.executable, "-m", "densecore_b200", "generate", "--model", stack.path, "--dtype", "float32", "--max-new", "6", "--max-ctx", "128"],
                       input="\n".join(",".join(map(str, p)) for p in ps), capture_output=True, text=True, timeout=300, cwd=root)
    assert r.returncode == 0, r.stderr
    assert [[int(t) for t in ln.split()] for ln in r.stdout.splitlines()] == [R.greedy(stack.cfg, stack.tensors, p, 6) for p in ps]


@pytest.mark.parametrize("n", [300, 700])
def test_large_products(ctx, tmp_path, n):
    """Enough rows and tokens for the wide tensor-core tiles (more tiles than SMs at the larger size), odd edges included."""
    c = Case(tmp_path, config([mamba(heads=20, vdim=40, state=16, groups=2, norm_groups=2), delta(heads=8, dim=32, vdim=64)], width=776, vocab=300, ff=[6500, 3000]),
             n=n, seed=3)
    m = c.model(ctx, "bfloat16", max_seqs=1, max_ctx=1024)
    assert close(run(m, c.tokens, [n]), c.want, "bfloat16")
    m.close()
