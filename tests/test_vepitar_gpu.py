"""Vepitar decoders through the library against the plain float64 restatement (oracle/layers_ref.py): every mechanism alone,
prompts in portions, mixed batches, reused pages and slots, window edges, long memory, long decoding, greedy generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import densecore_b200 as dc
from oracle import layers_ref as R
from stack_util import TOL, bf16_round, close, rel, run, write_model
from vepitar_util import Case, attention, config, dense, general, make_tensors, moe, planted_key_case, planted_state_case, shapes

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])

STACK = [attention(heads=4, kv_heads=4, dim=16, vdim=40, conv=3, window=70), general(), general(heads=5, dim=40), attention(), general(heads=1, dim=70),
         attention(heads=9, kv_heads=1, dim=36, vdim=20, conv=6, window=9)]
FEED = [dense(), moe(), None, moe(12, 4, 51), moe(5, 1, 33), dense(90)]


@pytest.fixture(scope="module")
def stack(tmp_path_factory):
    return Case(tmp_path_factory.mktemp("stack"), config(STACK, FEED))


ALONE = {
    "general": [general()],
    "general_one_head": [general(heads=1, dim=8)],
    "general_of_one": [general(heads=4, dim=1)],
    "general_odd_sizes": [general(heads=5, dim=19)],
    "general_32": [general(heads=5, dim=32)],
    "general_64": [general(heads=3, dim=64)],
    "general_100": [general(heads=2, dim=100)],
    "general_128": [general(heads=2, dim=128)],
    "general_200": [general(heads=1, dim=200)],
    "general_many_heads": [general(heads=21, dim=12)],
    "general_twice": [general(heads=2, dim=20), general(heads=7, dim=9)],
    "attention": [attention()],
    "attention_one_head": [attention(heads=1, kv_heads=1, dim=8, vdim=8)],
    "attention_of_one": [attention(heads=2, kv_heads=1, dim=1, vdim=1, scale=1.0)],
    "attention_every_head_its_own": [attention(heads=3, kv_heads=3, dim=16, vdim=16)],
    "attention_many_heads_one_key_head": [attention(heads=11, kv_heads=1, dim=20, vdim=12)],
    "attention_odd_sizes": [attention(heads=4, kv_heads=2, dim=17, vdim=13)],
    "attention_small_values": [attention(heads=4, kv_heads=2, dim=64, vdim=24, window=50)],
    "attention_small_keys": [attention(heads=4, kv_heads=2, dim=24, vdim=64, window=33)],
    "attention_64": [attention(heads=4, kv_heads=1, dim=64, vdim=64, window=65)],
    "attention_96": [attention(heads=2, kv_heads=1, dim=90, vdim=96, window=40)],
    "attention_128": [attention(heads=4, kv_heads=2, dim=128, vdim=128, window=70)],
    "attention_200_256": [attention(heads=2, kv_heads=1, dim=200, vdim=256, window=30)],
    "one_tap": [attention(conv=1)],
    "two_taps": [attention(conv=2)],
    "three_taps": [attention(conv=3, dim=33)],
    "five_taps": [attention(conv=5)],
    "sixteen_taps": [attention(conv=16, heads=3, kv_heads=1)],
    "taps_of_wide_heads": [attention(conv=7, heads=2, kv_heads=1, dim=150, vdim=140)],
    "window_one": [attention(window=1)],
    "window_two": [attention(window=2)],
    "window_of_a_page": [attention(window=16)],
    "window_beyond_the_context": [attention(window=5000)],
    "no_window": [attention(window=None)],
    "large_scale": [attention(scale=3.0)],
    "several_windows": [attention(window=5, conv=2), attention(window=60), attention(window=5)],
}


@pytest.mark.parametrize("name", list(ALONE))
@BOTH
def test_mechanism_alone(ctx, tmp_path, name, dtype):
    """One mixer without a feed-forward: the whole prompt at once, in sixteens, two at a time, and one by one at the end."""
    c = Case(tmp_path, config(ALONE[name], width=72, vocab=131, streams=2), n=140, seed=len(name))
    m = c.model(ctx, dtype)
    for cuts in ([140], [16], [2, 31, 5], [100, 1]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
    m.close()


@pytest.mark.parametrize("rank", [1, 8, 13, 64, 150])
@BOTH
def test_rank_of_the_decay(ctx, tmp_path, rank, dtype):
    c = Case(tmp_path, config([general(heads=2, dim=28)], width=72, vocab=131), n=70, seed=rank, rank=rank)
    m = c.model(ctx, dtype)
    for cuts in ([70], [1], [5, 2, 30]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
    m.close()


EXPERTS = {
    "some": moe(),
    "one": moe(1, 1, 24),
    "all_of_them": moe(6, 6, 24),
    "one_of_many": moe(12, 1, 20),
    "odd_size": moe(7, 2, 37),
    "tiny": moe(4, 2, 1),
    "long_rows": moe(4, 2, 700),
    "many": moe(136, 8, 16),
    "many_each": moe(40, 30, 24),
    "dense": dense(),
    "dense_odd": dense(37),
    "dense_of_one": dense(1),
    "dense_long": dense(500),
}


@pytest.mark.parametrize("name", list(EXPERTS))
@BOTH
def test_feed_forward_alone(ctx, tmp_path, name, dtype):
    """A mixer that adds nothing, then the feed-forward: one, a few, sixteen and many tokens in a step, and one-token steps of
    several sequences that share experts."""
    mlp = EXPERTS[name]
    cfg = config([attention(heads=1, kv_heads=1, dim=4, vdim=4)], mlp, width=mlp.get("router", {"experts": 0})["experts"] + 53, vocab=97)
    t = make_tensors(cfg, len(name))
    t["l0.mix.o"] *= 0
    c = Case(tmp_path, cfg, n=90, seed=3, tensors=t)
    m = c.model(ctx, dtype, max_seqs=16, max_ctx=128)
    for cuts in ([90], [1], [16], [8, 2, 17, 3]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
    for n in (2, 9, 16):
        seqs = [m.seq_alloc() for _ in range(n)]
        lg = np.stack([m.forward_batch([(s, c.tokens[j:j + 1]) for s, j in zip(seqs, range(i, 90, 90 // n))], np.arange(n)) for i in range(3)])
        want = np.stack([c.want[[j for _, j in zip(seqs, range(i, 90, 90 // n))]] for i in range(3)])    # a token's logits hang on it alone
        assert close(lg.reshape(3 * n, -1), want.reshape(3 * n, -1), dtype), n
        for s in seqs:
            m.seq_free(s)
    m.close()


@pytest.mark.parametrize("streams", range(1, 9))
@BOTH
def test_streams_and_odd_widths(ctx, tmp_path, dtype, streams):
    c = Case(tmp_path, config([general(heads=2, dim=10), attention(heads=2, kv_heads=1, dim=9, vdim=7, window=9), general(heads=1, dim=13)],
                              [moe(4, 2, 19), dense(21), None], width=51, vocab=77, eps=1e-2, streams=streams, mult=1.0 if streams == 3 else 0.35), n=48)
    m = c.model(ctx, dtype)
    for cuts in ([48], [1], [20, 2, 3]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
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
    """A one-token prompt and 330 decoded tokens: windows and pages pass over decoded keys."""
    c = Case(tmp_path, config(STACK[:4], [moe(), dense(), moe(), None]), n=331, seed=9)
    m = c.model(ctx, dtype, max_seqs=1)
    assert close(run(m, c.tokens, [1]), c.want, dtype)
    m.close()


# ---------------------------------------------------------------- keys and states that stand out
def cut_variants(n):
    return [n], [n - 1, 1], [n - 2, 2], [n - 18, 18], [max(1, n // 2 - 3), n]


STANDOUT = dict(heads=4, kv_heads=2, dim=40, vdim=24, conv=4)


@BOTH
@pytest.mark.parametrize("window,distance", [(33, 32), (33, 33), (64, 63), (64, 64), (100, 99), (100, 100), (48, 47), (48, 48), (300, 299), (300, 300),
                                             (129, 128), (129, 129), (300, 16), (300, 17), (2, 1), (2, 2)])
def test_last_key_inside_and_first_outside_the_window(ctx, tmp_path, window, distance, dtype):
    """Seen from a prompt (one step, and a short last portion) and from a decoded token."""
    n = distance + 20
    cfg, t, tokens, path = planted_key_case(tmp_path, attention(window=window, scale=0.45, **STANDOUT), n - 1 - distance, n)
    want = R.Stepper(cfg, t).step(tokens)[-1]
    if distance in (window, window - 1):
        cfg["layers"][0]["mixer"]["mask"]["size"] = window + (1 if distance == window else -1)
        assert rel(R.Stepper(cfg, t).step(tokens)[-1][None], want[None])[0] > 0.3       # one token more or less in the window shows
    m = dc.Model.from_dir(ctx, path, dtype, 2, 512)
    m.finalize()
    for cuts in cut_variants(n):
        assert rel(run(m, tokens, cuts)[-1:], want[None])[0] < TOL[dtype][1], cuts
    m.close()


@BOTH
def test_a_far_key_among_hundreds(ctx, tmp_path, dtype):
    """The standing-out key at every offset of a page, from the first token of the sequence on, decoded and in a portion."""
    for at in list(range(0, 34)) + [255, 256, 399]:
        cfg, t, tokens, path = planted_key_case(tmp_path, attention(window=1000, scale=0.45, **STANDOUT), at, 421)
        want = R.Stepper(cfg, t).step(tokens)[-1]
        if at in (0, 17):
            other = tokens.copy()
            other[at] = 0
            assert rel(R.Stepper(cfg, t).step(other)[-1][None], want[None])[0] > 0.3
        m = dc.Model.from_dir(ctx, path, dtype, 1, 512)
        m.finalize()
        cuts = [[421], [420, 1], [380, 41]][at % 3]
        assert rel(run(m, tokens, cuts)[-1:], want[None])[0] < TOL[dtype][1], at
        m.close()


@BOTH
@pytest.mark.parametrize("dim", [24, 40, 64, 130])
def test_what_the_state_remembers(ctx, tmp_path, dim, dtype):
    """A value stored hundreds of tokens ago, at every place of a block, is read back: in one step, over portions, decoded."""
    for at in list(range(0, 18)) + [31, 32, 200]:
        cfg, t, tokens, path = planted_state_case(tmp_path, dim, at, 260)
        want = R.Stepper(cfg, t).step(tokens)[-1]
        if at == 3:
            other = tokens.copy()
            other[at] = 0
            assert rel(R.Stepper(cfg, t).step(other)[-1][None], want[None])[0] > 0.3
        m = dc.Model.from_dir(ctx, path, dtype, 1, 512)
        m.finalize()
        cuts = [[260], [259, 1], [100, 2, 33, 5], [17, 1]][at % 4]
        assert rel(run(m, tokens, cuts)[-1:], want[None])[0] < TOL[dtype][1], at
        m.close()


@BOTH
@pytest.mark.parametrize("w0,bias", [(30.0, 30.0), (-30.0, 30.0), (30.0, -30.0), (-30.0, -30.0), (0.0, 0.0)])
def test_extreme_decays_and_removal_rates(ctx, tmp_path, w0, bias, dtype):
    """Decays at both of their bounds, keys that are removed at once and never."""
    cfg = config([general(heads=2, dim=36), general(heads=3, dim=20)], width=72, vocab=131)
    t = make_tensors(cfg, 2)
    for i in range(2):
        t[f"l{i}.mix.w0"], t[f"l{i}.mix.a.b"] = 0 * t[f"l{i}.mix.w0"] + w0, 0 * t[f"l{i}.mix.a.b"] + bias
    c = Case(tmp_path, cfg, n=150, tensors=t)
    m = c.model(ctx, dtype)
    for cuts in ([150], [1], [33, 2, 16]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
    m.close()


@BOTH
@pytest.mark.parametrize("pb", [-9.0, 0.0, 9.0])
def test_weights_do_not_sum_to_one(ctx, tmp_path, pb, dtype):
    """All keys nearly unseen, and all of them counted in full."""
    cfg = config([attention(window=60)], width=72, vocab=131, mult=0.05 if pb >= 0 else 20.0)
    t = make_tensors(cfg, 2)
    t["l0.mix.pb"] = bf16_round(t["l0.mix.pb"] + 2 + pb)
    c = Case(tmp_path, cfg, n=140, tensors=t)
    m = c.model(ctx, dtype)
    for cuts in ([140], [1], [33, 2, 16]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
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


@BOTH
def test_runs_repeat_bitwise(ctx, stack, dtype):
    m = stack.model(ctx, dtype)
    first = run(m, stack.tokens, [100, 3, 1])
    assert np.array_equal(first, run(m, stack.tokens, [100, 3, 1]))
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
def test_residual_after_every_layer_run(ctx, stack, dtype):
    _, layers = R.forward(stack.cfg, stack.tensors, stack.tokens[:21])
    m = stack.model(ctx, dtype)
    m.set_option("capture_layer_inputs", 1)
    s = m.seq_alloc()
    for a, b in ((0, 16), (16, 20), (20, 21)):
        m.forward_chunk(s, stack.tokens[a:b])
        for i in range(len(layers)):
            got = m.read_layer_input(i + 1, b - a)
            assert np.abs(got - layers[i, a:b]).max() < (1e-4 if dtype == "float32" else 0.2) * np.abs(layers[i]).std(), (a, i)
    m.close()


def test_forks(ctx, stack):
    """A fork shares pages and copies the recurrent state and the convolutions' inputs; both go on as if alone."""
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
        m.seq_truncate(b, 50)
    m.seq_truncate(b, 0)
    assert close(m.forward_batch([(b, stack.tokens[:40])], np.arange(40)), stack.want[:40], "float32")
    m.close()


def test_profile_and_stats(ctx, stack):
    m = stack.model(ctx, "bfloat16")
    s = m.seq_alloc()
    t = m.prefill(s, stack.tokens[:40])
    prof = m.profile_step([s], [t])
    assert {"mixer_in", "mixer_out", "mixer_gqa", "mixer_general_delta", "pre_norm", "router_topk", "moe_down", "ffn_down", "lm_head_argmax"} <= set(prof)
    launches, wbytes, kvb = m.step_stats()
    assert launches > 20 and wbytes > 0 and kvb > 0
    m.close()


def test_random_weights_from_a_config(ctx):
    cfg = config(STACK, FEED)
    m = dc.Model.from_config(ctx, cfg, shapes(cfg), max_seqs=1, max_ctx=128)
    m.init_synthetic(5, 0.05)
    m.finalize()
    s = m.seq_alloc()
    _, lg = m.prefill(s, np.arange(50), want_logits=True)
    assert np.isfinite(lg).all() and lg.std() > 0
    m.close()


def test_loading_errors(ctx, tmp_path):
    cfg = config([attention(), general()], [moe(4, 2, 12), dense(14)])
    t = make_tensors(cfg)

    def load(name, c=cfg, tensors=t, **kw):
        m = dc.Model.from_dir(ctx, write_model(tmp_path / name, c, tensors, **kw))
        try:
            m.finalize()
        finally:
            m.close()

    def changed(layer, part="mixer", **kw):
        c = json.loads(json.dumps(cfg))
        c["layers"][layer][part].update(kw)
        return c
    load("good")
    load("f32_vectors", f32=("l0.norm1", "l1.mix.w0", "l0.mix.pb", "l0.hc1.mix", "l0.mix.q.conv"))
    none = dict(cfg, layers=[dict(cfg["layers"][0], mlp=None), cfg["layers"][1]])
    load("unused", none, {k: v for k, v in t.items() if not k.startswith("l0.mlp.")})      # the second sublayer's norm and coefficients stay
    without = lambda *names: {k: v for k, v in t.items() if k not in names}
    for name, c, tensors, msg in (
            ("missing", cfg, without("l0.mlp.e3.up"), "l0.mlp.e3.up"),
            ("missing_gate", cfg, without("l0.mix.g"), "l0.mix.g"),
            ("missing_rank", cfg, without("l1.mix.w1"), "l1.mix.w1"),
            ("missing_hyper", cfg, without("l1.hc2.mix"), "l1.hc2.mix"),
            ("extra", cfg, dict(t, **{"l0.mlp.e0.gate": t["l0.mlp.e3.up"]}), "l0.mlp.e0.gate"),
            ("head", cfg, dict(t, head=t["embed"]), "head"),
            ("shape", cfg, dict(t, embed=t["embed"][:-1]), "embed"),
            ("mixer", dict(cfg, layers=[dict(cfg["layers"][0], type="lightning")] + cfg["layers"][1:]), t, "lightning"),
            ("kind", changed(0, "mlp", kind="sparse"), t, "kind"),
            ("heads", changed(0, kv_heads=4), t, "kv_heads"),
            ("taps", changed(0, conv=0), t, "conv"),
            ("no_taps", changed(0, conv=None), t, "conv"),
            ("no_scale", changed(0, scale=None), t, "scale"),
            ("window", changed(0, mask={"size": 0}), t, "size"),
            ("dim", changed(1, dim=300), t, "dim"),
            ("streams", dict(cfg, streams=9), t, "streams"),
            ("no_streams", {k: v for k, v in cfg.items() if k != "streams"}, t, "streams"),
            ("no_mult", {k: v for k, v in cfg.items() if k != "residual_mult"}, t, "residual_mult"),
            ("loop", dict(cfg, loop={"start": 0, "stop": 1, "times": 2}), t, "loop"),
            ("too_few", changed(0, "mlp", router={"experts": 4, "top": 5}), t, "top")):
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
    """Enough rows, experts and tokens for the wide tensor-core tiles: runs of more and of fewer than 128 tokens, odd edges."""
    layers = [general(heads=10, dim=64), attention(heads=16, kv_heads=2, dim=64, vdim=48, window=200), general(heads=7, dim=48)]
    c = Case(tmp_path, config(layers, [moe(3, 2, 1100), moe(24, 4, 150), dense(1300)], width=776, vocab=300), n=n, seed=3, rank=40)
    m = c.model(ctx, "bfloat16", max_seqs=1, max_ctx=1024)
    assert close(run(m, c.tokens, [n]), c.want, "bfloat16")
    assert close(run(m, c.tokens[:n // 2], [n // 2 - 20, 16, 1]), c.want[:n // 2], "bfloat16")
    m.close()
