"""Gomuzen decoders through the library against the plain float64 restatement (oracle/layers_ref.py): every mechanism
alone, prompts in portions, mixed batches, reused pages and slots, window edges, long decoding, greedy generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import densecore_b200 as dc
from gomuzen_util import YARN, Case, config, differential, kept, latent, make_tensors, moe, settled_tokens
from oracle import layers_ref as R
from stack_util import TOL, bf16_round, close, rel, run, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])

STACK = [kept(window=70, heads=4, kv_heads=4, dim=16, vdim=40, dims=10, scaling=None), latent(), differential(), kept(), differential(heads=3, kv_heads=1, dim=28, vdim=18, dims=28),
         latent(heads=2, dim=34, rot_dim=6, vdim=12, kv_rank=24)]
FEED = [moe(), moe(12, 4, 3, 2, 30, 0.8), None, moe(9, 2, 1, 1, 51), moe(8, 6, 4, 3, 24, 3.0, 0.6), moe(5, 1, 5, 2, 33)]


@pytest.fixture(scope="module")
def stack(tmp_path_factory):
    return Case(tmp_path_factory.mktemp("stack"), config(STACK, FEED, loop=(1, 4, 2)))


ALONE = {
    "latent": [latent()],
    "latent_odd_sizes": [latent(heads=5, dim=9, rot_dim=6, vdim=7, kv_rank=21)],
    "latent_wide_values": [latent(heads=2, dim=70, rot_dim=20, vdim=140, kv_rank=72)],
    "latent_long_rank": [latent(heads=2, dim=48, rot_dim=32, vdim=64, kv_rank=300)],
    "latent_many_heads": [latent(heads=17, dim=8, rot_dim=2, vdim=8, kv_rank=16)],
    "differential": [differential()],
    "differential_one_head": [differential(heads=1, kv_heads=1, dim=8, vdim=8, dims=2)],
    "differential_every_head_its_own": [differential(heads=3, kv_heads=3, dim=16, vdim=16, dims=16)],
    "differential_many_heads_one_key_head": [differential(heads=9, kv_heads=1, dim=20, vdim=12, dims=6)],
    "differential_odd_sizes": [differential(heads=4, kv_heads=2, dim=17, vdim=11, dims=6)],
    "differential_64_64": [differential(heads=4, kv_heads=2, dim=64, vdim=64, dims=32)],
    "differential_64_128": [differential(heads=4, kv_heads=2, dim=64, vdim=128, dims=64)],
    "differential_100_90": [differential(heads=2, kv_heads=1, dim=100, vdim=90, dims=40)],
    "differential_128_128": [differential(heads=2, kv_heads=1, dim=128, vdim=128, dims=64)],
    "differential_24_200": [differential(heads=2, kv_heads=2, dim=24, vdim=200, dims=8)],
    "differential_128_256": [differential(heads=3, kv_heads=1, dim=128, vdim=256, dims=128)],
    "differential_no_cap": [differential(softcap=None)],
    "differential_tight_cap": [differential(softcap=0.5)],
    "differential_diff_zero": [differential(diff=0.0)],
    "differential_large_diff": [differential(diff=0.9)],
    "differential_windowed": [differential(mask=(19, 2)), differential(mask=(40, 0), dim=64, vdim=128)],
    "kept": [kept()],
    "kept_one_head": [kept(heads=1, kv_heads=1, dim=8, vdim=8, dims=2)],
    "kept_many_heads_one_key_head": [kept(heads=9, kv_heads=1, dim=20, vdim=24, dims=6)],
    "kept_odd_sizes": [kept(heads=4, kv_heads=2, dim=17, vdim=13, dims=6, window=13)],
    "kept_32_64": [kept(heads=4, kv_heads=2, dim=32, vdim=64, dims=32, window=33, keep=5)],
    "kept_64_32": [kept(heads=4, kv_heads=2, dim=64, vdim=32, dims=20, window=50, keep=1)],
    "kept_96": [kept(heads=6, kv_heads=3, dim=96, vdim=80, dims=32, window=40)],
    "kept_64_128": [kept(heads=2, kv_heads=1, dim=56, vdim=128, dims=56, window=40)],
    "kept_128": [kept(heads=4, kv_heads=1, dim=128, vdim=128, dims=64, window=70)],
    "kept_200_256": [kept(heads=2, kv_heads=1, dim=200, vdim=256, dims=100, window=30)],
    "kept_none": [kept(keep=0)],
    "kept_more_than_the_window": [kept(window=5, keep=40)],
    "kept_across_tiles": [kept(window=20, keep=70)],
    "kept_window_one": [kept(window=1, keep=1)],
    "kept_no_window_but_the_first": [kept(window=1, keep=0)],
    "kept_whole_context": [kept(window=5000, keep=7)],
    "kept_no_cap": [kept(softcap=None)],
    "kept_tight_cap": [kept(softcap=0.7)],
    "kept_no_scaling": [kept(scaling=None, base=10000.0)],
    "kept_scaling_of_one": [kept(scaling=dict(YARN, factor=1.0))],
    "kept_steep_ramp": [kept(dims=20, base=50.0, scaling=dict(YARN, fast=2.0, slow=1.99))],
    "kept_windows_and_rotations": [kept(window=5, keep=1), kept(window=60, keep=9, base=30.0), kept(window=5, keep=2, scaling=dict(YARN, factor=2.0))],
}


@pytest.mark.parametrize("name", list(ALONE))
@BOTH
def test_mechanism_alone(ctx, tmp_path, name, dtype):
    """One mixer without a feed-forward: the whole prompt at once, in sixteens, two at a time, and one by one at the end."""
    c = Case(tmp_path, config(ALONE[name], width=72, vocab=131), n=140, seed=len(name))
    m = c.model(ctx, dtype)
    for cuts in ([140], [16], [2, 31, 5], [100, 1]):
        assert close(run(m, c.tokens, cuts), c.want, dtype), cuts
    m.close()


EXPERTS = {
    "some": (moe(), 0.0),
    "one": (moe(1, 1, 1, 1, 24), 0.0),
    "all_of_them": (moe(6, 6, 1, 1, 24), 0.0),
    "whole_groups": (moe(12, 6, 4, 2, 20), 0.0),
    "groups_of_one": (moe(6, 2, 6, 3, 20), 0.0),
    "every_group_kept": (moe(12, 3, 3, 3, 20), 0.0),
    "negative_choice_scores": (moe(12, 4, 3, 1, 20), -3.0),
    "odd_size": (moe(7, 2, 1, 1, 37), 0.0),
    "tiny": (moe(4, 2, 2, 1, 1), 0.0),
    "long_rows": (moe(4, 2, 2, 1, 700), 0.0),
    "tight_limit": (moe(limit=0.05), 0.0),
    "loose_limit": (moe(limit=50.0), 0.0),
    "small_scale": (moe(scale=0.1), 0.0),
    "many": (moe(136, 8, 8, 4, 16), 0.0),
    "as_many_groups_as_a_warp": (moe(96, 20, 32, 11, 8), 0.0),
}


@pytest.mark.parametrize("name", list(EXPERTS))
@BOTH
def test_experts_alone(ctx, tmp_path, name, dtype):
    """A mixer that adds nothing, then experts: one, a few, sixteen and many tokens in a step, and one-token steps of several
    sequences that share experts."""
    mlp, correction = EXPERTS[name]
    cfg = config([latent(heads=1, dim=4, rot_dim=2, vdim=4, kv_rank=8)], mlp, width=mlp["router"]["experts"] + 53, vocab=97)
    t = make_tensors(cfg, len(name), correction)
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


@pytest.mark.parametrize("loop", [None, (0, 3, 1), (0, 1, 4), (2, 3, 2), (0, 3, 2), (1, 2, 3)], ids=str)
@BOTH
def test_loops_and_odd_widths(ctx, tmp_path, dtype, loop):
    """Every pass has its own cache and vector, whatever the layers."""
    c = Case(tmp_path, config([differential(heads=2, kv_heads=1, dim=10, vdim=9, dims=4), latent(heads=2, dim=9, rot_dim=4, vdim=7, kv_rank=13), kept(heads=2, window=9, keep=2)],
                              [moe(4, 2, 2, 1, 19), None, moe(6, 2, 2, 1, 21)], width=51, vocab=77, eps=1e-2, loop=loop), n=48)
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
    """A one-token prompt and 330 decoded tokens: windows and pages pass over decoded keys, the first ones stay in sight."""
    c = Case(tmp_path, config(STACK[:4], moe(), loop=(1, 3, 2)), n=331, seed=9)
    m = c.model(ctx, dtype, max_seqs=1)
    assert close(run(m, c.tokens, [1]), c.want, dtype)
    m.close()


# ---------------------------------------------------------------- keys that stand out
def planted_key_case(path, layer, at, n, seed=3):
    """One layer whose query of token B finds token A's key far above all others (with two maps: by the first map).  A
    occurs once, at place `at`, and B at the end, so the answer hangs on whether that one key is seen."""
    m, kind = layer["mixer"], layer["type"]
    cfg = config([layer], width=64, vocab=97)
    t = make_tensors(cfg, seed)
    A, B, eps, H = 95, 96, cfg["norm"]["eps"], m["heads"]
    P = {k[len("l0.mix."):]: v.astype(np.float64) for k, v in t.items() if k.startswith("l0.mix.")}
    h = R.rms_norm(t["embed"].astype(np.float64), t["l0.norm1"].astype(np.float64), eps)
    q = P["q"].reshape(H, -1, 64)
    bias = P["q.b"].reshape(H, -1) if "q.b" in P else np.zeros(q.shape[:2])
    if kind == "latent_attention":
        c = R.rms_norm(P["dkv"][:m["kv_rank"]] @ h[A], P["dkv.norm"], eps)
        target = (P["uk"] @ c).reshape(H, m["dim"])
    elif kind == "attention":
        k = R.rms_norm((P["k"] @ h[A]).reshape(m["kv_heads"], 2, m["dim"])[:, 0], P["k.norm"], eps)
        target = k[np.arange(H) // (H // m["kv_heads"])] / P["q.norm"]
    else:
        k = (P["k"] @ h[A] + P["k.b"]).reshape(m["kv_heads"], m["dim"])
        target = k[np.arange(H) // (H // m["kv_heads"])]
    if kind != "latent_attention":
        target[:, :m["rot"]["dims"]] = 0            # nothing of what is turned
    d = m["dim"]
    for i in range(H):                              # W_q h_B + b = target
        q[i, :d] += np.outer(target[i] - q[i, :d] @ h[B] - bias[i, :d], h[B] / (h[B] @ h[B]))
    t["l0.mix.q"] = bf16_round(q.reshape(-1, 64))
    tokens = np.random.default_rng(seed).integers(0, 95, size=n)
    tokens[-1], tokens[at] = B, A
    return cfg, t, tokens, write_model(path, cfg, t)


def cut_variants(n):
    return [n], [n - 1, 1], [n - 2, 2], [n - 18, 18], [max(1, n // 2 - 3), n]


STANDOUT = dict(heads=4, kv_heads=2, dim=48, vdim=40, dims=8, scale=0.36, softcap=40.0)


@BOTH
@pytest.mark.parametrize("form", ["kept", "differential"])
@pytest.mark.parametrize("window,distance", [(33, 32), (33, 33), (64, 63), (64, 64), (100, 99), (100, 100), (48, 47), (48, 48), (300, 299), (300, 300),
                                             (129, 128), (129, 129), (300, 16), (300, 17), (2, 1), (2, 2), (1, 1)])
def test_last_key_inside_and_first_outside_the_window(ctx, tmp_path, form, window, distance, dtype):
    """Seen from a prompt (one step, and a short last portion) and from a decoded token."""
    layer = kept(window=window, keep=3, scaling=None, **STANDOUT) if form == "kept" else differential(mask=(window, 3), **STANDOUT)
    n = distance + 20
    cfg, t, tokens, path = planted_key_case(tmp_path, layer, n - 1 - distance, n)
    want = R.Stepper(cfg, t).step(tokens)[-1]
    if distance == window or (window > 1 and distance == window - 1):
        cfg["layers"][0]["mixer"]["mask"]["size"] = window + (1 if distance == window else -1)
        assert rel(R.Stepper(cfg, t).step(tokens)[-1][None], want[None])[0] > 0.3       # one token more or less in the window shows
    m = dc.Model.from_dir(ctx, path, dtype, 2, 512)
    m.finalize()
    for cuts in cut_variants(n):
        assert rel(run(m, tokens, cuts)[-1:], want[None])[0] < TOL[dtype][1], cuts
    m.close()


@BOTH
@pytest.mark.parametrize("window,keep,at,n", [(21, 3, 2, 90), (21, 3, 3, 90), (21, 1, 0, 200), (21, 1, 1, 200), (70, 16, 15, 300), (70, 16, 16, 300), (40, 64, 63, 250),
                                              (40, 64, 64, 250), (40, 65, 64, 250), (1, 1, 0, 40), (1, 1, 1, 40), (30, 20, 19, 50), (30, 20, 20, 50), (30, 20, 19, 51),
                                              (30, 20, 20, 51)])
def test_last_kept_token_and_the_next(ctx, tmp_path, window, keep, at, n, dtype):
    layer = kept(window=window, keep=keep, scaling=None, **STANDOUT)
    cfg, t, tokens, path = planted_key_case(tmp_path, layer, at, n)
    want = R.Stepper(cfg, t).step(tokens)[-1]
    if n - 1 - at >= window:
        cfg["layers"][0]["mixer"]["mask"]["keep_first"] = keep + (-1 if at < keep else 1)
        assert rel(R.Stepper(cfg, t).step(tokens)[-1][None], want[None])[0] > 0.3
    m = dc.Model.from_dir(ctx, path, dtype, 2, 512)
    m.finalize()
    for cuts in cut_variants(n):
        assert rel(run(m, tokens, cuts)[-1:], want[None])[0] < TOL[dtype][1], cuts
    m.close()


FAR = {"latent": latent(heads=4, dim=48, rot_dim=8, vdim=40, kv_rank=60, scale=0.5), "differential": differential(**STANDOUT),
       "kept": kept(window=1000, keep=2, scaling=None, **STANDOUT)}


@BOTH
@pytest.mark.parametrize("form", list(FAR))
def test_a_far_key_among_hundreds(ctx, tmp_path, form, dtype):
    """The standing-out key at every offset of a page, from the first token of the sequence on, decoded and in a portion."""
    for at in list(range(0, 34)) + [255, 256, 399]:
        cfg, t, tokens, path = planted_key_case(tmp_path, FAR[form], at, 421)
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
@pytest.mark.parametrize("form", ["differential", "kept"])
def test_scores_far_above_the_cap(ctx, tmp_path, form, dtype):
    """Raw scores of hundreds that the cap brings down to a few: every visible key keeps a share."""
    sizes = dict(heads=2, kv_heads=1, dim=32, vdim=24, dims=4, scale=20.0, softcap=3.0)
    cfg = config([differential(**sizes) if form == "differential" else kept(window=40, scaling=None, **sizes)], width=64, vocab=61)
    c = Case(tmp_path, cfg, n=90, seed=4)
    free = json.loads(json.dumps(cfg))
    free["layers"][0]["mixer"]["softcap"] = None
    assert rel(R.Stepper(free, c.tensors).step(c.tokens), c.want).max() > 0.3
    m = c.model(ctx, dtype, max_ctx=128)
    for cuts in ([90], [1], [40, 7]):
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


def test_forks_and_cuts(ctx, stack):
    """A fork shares pages and both go on as if alone; a sequence can be cut back and go on."""
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
    m.seq_truncate(b, 50)
    assert close(m.forward_batch([(b, stack.tokens[50:90])], np.arange(40)), stack.want[50:90], "float32")
    m.close()


def test_profile_and_stats(ctx, stack):
    m = stack.model(ctx, "bfloat16")
    s = m.seq_alloc()
    t = m.prefill(s, stack.tokens[:40])
    prof = m.profile_step([s], [t])
    assert {"mixer_in", "mixer_out", "mixer_gqa", "mixer_latent", "pre_norm", "router_topk", "moe_down", "lm_head_argmax"} <= set(prof)
    launches, wbytes, kvb = m.step_stats()
    assert launches > 20 and wbytes > 0 and kvb > 0
    m.close()


def test_random_weights_from_a_config(ctx):
    m = dc.Model.from_config(ctx, config(STACK, FEED, loop=(0, 2, 2)), max_seqs=1, max_ctx=128)
    m.init_synthetic(5, 0.05)
    m.finalize()
    s = m.seq_alloc()
    _, lg = m.prefill(s, np.arange(50), want_logits=True)
    assert np.isfinite(lg).all() and lg.std() > 0
    m.close()


def test_loading_errors(ctx, tmp_path):
    cfg = config([latent(), differential(), kept()], moe(4, 2, 2, 1, 12), loop=(1, 3, 2))
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

    def routed(**kw):
        c = json.loads(json.dumps(cfg))
        c["layers"][1]["mlp"]["router"].update(kw)
        return c

    def looped(**kw):
        return dict(cfg, loop=dict(cfg["loop"], **kw))
    load("good")
    load("f32_vectors", f32=("l0.norm1", "l1.mlp.correction", "loop.step", "l1.mix.lq1"))
    for name, c, tensors, msg in (
            ("missing", cfg, {k: v for k, v in t.items() if k != "l1.mlp.e3.up"}, "l1.mlp.e3.up"),
            ("missing_gate", cfg, {k: v for k, v in t.items() if k != "l0.mix.g"}, "l0.mix.g"),
            ("extra", cfg, dict(t, **{"l1.mlp.e4.up": t["l1.mlp.e3.up"]}), "l1.mlp.e4.up"),
            ("shape", cfg, dict(t, head=t["head"][:-1]), "head"),
            ("mixer", dict(cfg, layers=[dict(cfg["layers"][0], type="lightning")] + cfg["layers"][1:]), t, "lightning"),
            ("kind", changed(0, "mlp", kind="dense"), t, "kind"),
            ("heads", changed(1, kv_heads=3), t, "kv_heads"),
            ("diff", changed(1, diff=None), t, "diff"),
            ("cap", changed(1, softcap=-1.0), t, "softcap"),
            ("keep", changed(2, mask={"size": 4, "keep_first": -1}), t, "keep_first"),
            ("latent_keep", changed(0, mask={"size": 4, "keep_first": 1}), t, "keep_first"),
            ("rotation", changed(2, rot={"base": 100.0, "dims": 26}), t, "dims"),
            ("groups", routed(groups={"count": 3, "keep": 1}), t, "groups.count"),
            ("too_few", routed(top=3), t, "top"),
            ("limit", changed(0, "mlp", expert={"ff": 12}), t, "limit"),
            ("loop_stop", looped(stop=4), t, "stop"),
            ("loop_start", looped(start=3), t, "start"),
            ("loop_times", looped(times=3), t, "loop.step")):
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
    layers = [latent(heads=6, dim=40, rot_dim=24, vdim=48, kv_rank=136), differential(heads=8, kv_heads=2, dim=48, vdim=96, dims=20), kept(heads=16, kv_heads=2, dim=48, vdim=48, dims=20, window=200)]
    c = Case(tmp_path, config(layers, [moe(3, 2, 1, 1, 1100), moe(24, 4, 4, 2, 150), None], width=776, vocab=300), n=n, seed=3)
    m = c.model(ctx, "bfloat16", max_seqs=1, max_ctx=1024)
    assert close(run(m, c.tokens, [n]), c.want, "bfloat16")
    assert close(run(m, c.tokens[:n // 2], [n // 2 - 20, 16, 1]), c.want[:n // 2], "bfloat16")
    m.close()
