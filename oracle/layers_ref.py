"""Plain, slow restatement of the layer-list decoders' mechanisms in float64 numpy, one function per mechanism.

TEST INFRASTRUCTURE ONLY: shares no code with the product path.  A model is (config dict, {name: ndarray});
`forward` runs one whole sequence and returns logits and the residual after every layer; `Stepper` runs the same
layers with carried state, any number of tokens at a time.
"""
from __future__ import annotations

import numpy as np

F = np.float64


# ---------------------------------------------------------------- elementwise and norms
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    """Over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def unit_vectors(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def linear(x, w):
    """x [T, K], w [N, K]."""
    return x @ w.T


# ---------------------------------------------------------------- time mixing pieces
def short_conv(x, w, bias=None, history=None):
    """Causal per-channel convolution over time: x [T, C], w [C, taps] (last column: the current token).
    history [taps - 1, C]: the inputs before x (zeros at the start).  Returns (y, the new history)."""
    T, taps = x.shape[0], w.shape[1]
    if history is None:
        history = np.zeros((taps - 1, x.shape[1]), F)
    xx = np.concatenate([history, x], axis=0)
    y = np.zeros_like(x)
    for j in range(taps):
        y += xx[j:j + T] * w[:, j]
    if bias is not None:
        y = y + bias
    return y, xx[xx.shape[0] - (taps - 1):]


def rotate_interleaved(x, pos, dims, base):
    """x [T, H, D]: the first `dims` dimensions of every head turned by the position, pairs (2i, 2i + 1)."""
    out = x.copy()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def delta_rule(q, k, v, beta, g, S):
    """Gated delta rule, token by token.  q, k, g [T, H, d]; v [T, H, e]; beta [T, H]; S [H, d, e] (changed in
    place).  Returns o [T, H, e]."""
    T, H = beta.shape
    o = np.zeros((T, H, v.shape[2]), F)
    for t in range(T):
        for h in range(H):
            S[h] = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] = S[h] + np.outer(k[t, h], u)
            o[t, h] = S[h].T @ q[t, h]
    return o


def ssd_scan(x, B, C, dt, A_log, D, S):
    """x [T, H, e]; B, C [T, G, n]; dt [T, H] (after softplus); S [H, n, e] (changed in place).  y [T, H, e]."""
    T, H, _ = x.shape
    per = H // B.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for h in range(H):
            b, c = B[t, h // per], C[t, h // per]
            S[h] = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(b, x[t, h])
            y[t, h] = S[h].T @ c + D[h] * x[t, h]
    return y


def windowed_softmax(scores, i, window, sink=None, keep=0):
    """scores over keys 0 .. i -> weights; keys with i - j >= window are not seen, except the first `keep` of the
    sequence.  sink: score of one more term of the denominator that has no value."""
    n = scores.shape[-1]
    seen = ((i - np.arange(n)) < window) | (np.arange(n) < keep) if window else np.ones(n, bool)
    s = np.where(seen, scores, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    s = np.exp(s - top)
    return s / (s.sum(axis=-1, keepdims=True) + (0.0 if sink is None else np.exp(sink - top)))


def yarn_frequencies(dims, base, scaling=None):
    """(angle per position of every pair, factor of cos and sin).  scaling: {factor, original, fast, slow}; pairs that
    turn less than `slow` times over the original context are slowed down by the factor, those that turn more than
    `fast` times are left alone, with a linear ramp over the pairs between."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], F)
    if not scaling:
        return f, 1.0
    pair_of = lambda turns: dims * np.log(scaling["original"] / (2 * np.pi * turns)) / (2 * np.log(base))
    lo = max(np.floor(pair_of(scaling["fast"])), 0)
    hi = min(np.ceil(pair_of(scaling["slow"])), dims - 1)
    slowed = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0, 1)
    return f * (1 - slowed) + f / scaling["factor"] * slowed, 0.1 * np.log(scaling["factor"]) + 1.0


def rotate_pairs(x, pos, freq, mul):
    """x [T, H, D]: pairs (2i, 2i + 1) of the first 2 len(freq) dimensions turned by pos * freq[i] and scaled."""
    out = x.copy()
    for i, f in enumerate(freq):
        c, s = mul * np.cos(pos * f)[:, None], mul * np.sin(pos * f)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def rotate_halves(x, pos, freq, mul):
    """x [T, H, D]: pairs (i, i + n) of the first 2 n dimensions (n frequencies) turned by pos * freq[i] and scaled."""
    out, n = x.copy(), len(freq)
    for i, f in enumerate(freq):
        c, s = mul * np.cos(pos * f)[:, None], mul * np.sin(pos * f)[:, None]
        u, v = x[:, :, i], x[:, :, i + n]
        out[:, :, i] = u * c - v * s
        out[:, :, i + n] = v * c + u * s
    return out


def soft_cap(scores, cap):
    return cap * np.tanh(scores / cap)


def paged_attention(q, k, v, pos, scale, cap=None, window=None, keep=0):
    """q [T, H, d] over every earlier key k [n, G, d] and value v [n, G, e]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    of = np.arange(H) // (H // k.shape[1])
    out = np.zeros((T, H, v.shape[2]), F)
    for t in range(T):
        n = int(pos[t]) + 1
        s = np.einsum("hd,nhd->hn", q[t], k[:n, of]) * scale
        if cap:
            s = soft_cap(s, cap)
        out[t] = np.einsum("hn,nhe->he", windowed_softmax(s, n - 1, window, keep=keep), v[:n, of])
    return out


def grow(st, **new):
    """Appends rows to the cached arrays and returns them whole."""
    for n, a in new.items():
        st[n] = np.concatenate([st[n], a]) if n in st else a
    return [st[n] for n in new]


def decayed_linear_attention(q, k, v, decay, S):
    """S <- decay S + k v^T, o = S^T q, token by token.  q, k [T, H, d]; v [T, H, e]; decay [H]; S [H, d, e] (changed
    in place).  Returns o [T, H, e]."""
    o = np.zeros_like(v)
    for t in range(q.shape[0]):
        for h in range(q.shape[1]):
            S[h] = decay[h] * S[h] + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o


# ---------------------------------------------------------------- mixers
def mix_channel_delta(h, P, m, eps, st):
    T, H, KH, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    z = {}
    for n in "qkv":
        y, st["conv." + n] = short_conv(linear(h, P[n]), P[n + ".conv"], None, st.get("conv." + n))
        z[n] = silu(y)
    of = np.arange(H) // (H // KH)
    q = unit_vectors(z["q"].reshape(T, KH, d))[:, of] * d ** -0.5
    k = unit_vectors(z["k"].reshape(T, KH, d))[:, of]
    v = z["v"].reshape(T, H, e)
    beta = sigmoid(linear(h, P["b"]))
    raw = linear(linear(h, P["a1"]), P["a2"]) + P["dt_bias"].reshape(-1)
    g = np.exp(-np.exp(P["A_log"].reshape(-1))[None, :, None] * softplus(raw).reshape(T, H, d))
    if "S" not in st:
        st["S"] = np.zeros((H, d, e), F)
    o = delta_rule(q, k, v, beta, g, st["S"])
    o = rms_norm(o, P["norm"], eps) * sigmoid(linear(linear(h, P["g1"]), P["g2"])).reshape(T, H, e)
    return linear(o.reshape(T, H * e), P["o"])


def mix_mamba2(h, P, m, eps, st):
    T, H, e, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * e
    z, xbc, dt = np.split(linear(h, P["in"]), [inner, 2 * inner + 2 * G * N], axis=1)
    y, st["conv"] = short_conv(xbc, P["conv"], P["conv.b"], st.get("conv"))
    x, B, C = np.split(silu(y), [inner, inner + G * N], axis=1)
    dt = softplus(dt + P["dt_bias"].reshape(-1))
    if "S" not in st:
        st["S"] = np.zeros((H, N, e), F)
    y = ssd_scan(x.reshape(T, H, e), B.reshape(T, G, N), C.reshape(T, G, N), dt, P["A_log"].reshape(-1), P["D"].reshape(-1), st["S"])
    y = y.reshape(T, inner) * silu(z)
    ng = m["norm_groups"]
    y = rms_norm(y.reshape(T, ng, inner // ng), 1.0, eps).reshape(T, inner) * P["norm"]
    return linear(y, P["o"])


def mix_latent_attention(h, P, m, eps, pos, cache):
    """cache: {"c": [n, kv_rank], "r": [n, rot_dim]} holding every token up to and including these (see
    latent_append)."""
    T, H, d, r, e = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = linear(h, P["q"]).reshape(T, H, d + r)
    qu, qr = q[:, :, :d], rotate_interleaved(q[:, :, d:], pos, m["rot"]["dims"], m["rot"]["base"])
    c, kr = cache["c"], cache["r"]
    ku = linear(c, P["uk"]).reshape(-1, H, d)
    v = linear(c, P["uv"]).reshape(-1, H, e)
    window = (m.get("mask") or {}).get("size")
    out = np.zeros((T, H, e), F)
    for t in range(T):
        n = int(pos[t]) + 1
        s = (np.einsum("hd,nhd->hn", qu[t], ku[:n]) + np.einsum("hr,nr->hn", qr[t], kr[:n])) * m["scale"]
        out[t] = np.einsum("hn,nhe->he", windowed_softmax(s, n - 1, window), v[:n])
    if "g" in P:                # one gate per head
        out = out * sigmoid(linear(h, P["g"]))[:, :, None]
    return linear(out.reshape(T, H * e), P["o"])


def latent_append(h, P, m, eps, pos, cache):
    kv = linear(h, P["dkv"])
    c = rms_norm(kv[:, :m["kv_rank"]], P["dkv.norm"], eps)
    kr = rotate_interleaved(kv[:, None, m["kv_rank"]:], pos, m["rot"]["dims"], m["rot"]["base"])[:, 0]
    if "c" in cache:
        c, kr = np.concatenate([cache["c"], c]), np.concatenate([cache["r"], kr])
    cache["c"], cache["r"] = c, kr


def dense_mlp(h, P):
    return linear(gelu_tanh(linear(h, P["gate"])) * linear(h, P["up"]), P["down"])


def mix_attention(h, P, m, eps, pos, st):
    """Grouped-query attention whose values are the raw keys; a sink of score 0.  st: {"k", "v"} of earlier tokens."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = linear(h, P["q"]) + P["q.b"]
    v = linear(h, P["k"]) + P["k.b"]
    freq, mul = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = rotate_pairs(rms_norm(q, P["q.norm"], eps).reshape(T, H, d), pos, freq, mul)
    k = rotate_pairs(rms_norm(v, P["k.norm"], eps).reshape(T, G, d), pos, freq, mul)
    v = v.reshape(T, G, d)
    if "k" in st:
        k, v = np.concatenate([st["k"], k]), np.concatenate([st["v"], v])
    st["k"], st["v"] = k, v
    of = np.arange(H) // (H // G)
    out = np.zeros((T, H, d), F)
    for t in range(T):
        n = int(pos[t]) + 1
        s = np.einsum("hd,nhd->hn", q[t], k[:n, of]) * m["scale"]
        out[t] = np.einsum("hn,nhd->hd", windowed_softmax(s, n - 1, m["mask"]["size"], sink=0.0), v[:n, of])
    return linear(out.reshape(T, H * d), P["o"]) + P["o.b"]


def mix_lightning(h, P, m, eps, st):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (silu(linear(h, P[n])).reshape(T, H, d) for n in "qk")
    v = silu(linear(h, P["v"])).reshape(T, H, e)
    if "S" not in st:
        st["S"] = np.zeros((H, d, e), F)
    o = decayed_linear_attention(q, k, v, np.array(m["decay"], F), st["S"]).reshape(T, H * e)
    return linear(rms_norm(o, P["norm"], eps) * sigmoid(linear(h, P["g"])), P["o"])


def clamped_mlp(h, P, limit):
    g = np.minimum(linear(h, P["gate"]), limit)
    u = np.clip(linear(h, P["up"]), -limit, limit)
    return linear(g * sigmoid(1.702 * g) * (u + 1), P["down"])


def mix_differential(h, P, m, eps, pos, st):
    """Two attention maps per head over the same values; the second is taken off, weighted by one learned number."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freq, mul = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = rotate_halves(rms_norm(linear(h, P["q"]).reshape(T, H * 2, d), P["q.norm"], eps), pos, freq, mul).reshape(T, H, 2, d)
    k = rotate_halves(rms_norm(linear(h, P["k"]).reshape(T, G * 2, d), P["k.norm"], eps), pos, freq, mul).reshape(T, G, 2, d)
    k, v = grow(st, k=k, v=linear(h, P["v"]).reshape(T, G, e))
    mask = m.get("mask") or {}
    a1, a2 = (paged_attention(q[:, :, i], k[:, :, i], v, pos, m["scale"], m.get("softcap"), mask.get("size"), mask.get("keep_first", 0)) for i in range(2))
    lam = np.exp(np.sum(P["lq1"] * P["lk1"])) - np.exp(np.sum(P["lq2"] * P["lk2"])) + m["diff"]
    o = rms_norm(a1 - lam * a2, 1.0, eps) * (1.0 - m["diff"])
    return linear(o.reshape(T, H * e), P["o"])


def mix_kept_window(h, P, m, eps, pos, st):
    """Grouped-query attention with biased projections over a sliding window and the first tokens of the sequence."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (linear(h, P[n]) + P[n + ".b"] for n in "qkv")
    freq, mul = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = rotate_halves(q.reshape(T, H, d), pos, freq, mul)
    k, v = grow(st, k=rotate_halves(k.reshape(T, G, d), pos, freq, mul), v=v.reshape(T, G, e))
    mask = m.get("mask") or {}
    o = paged_attention(q, k, v, pos, m["scale"], m.get("softcap"), mask.get("size"), mask.get("keep_first", 0))
    return linear(o.reshape(T, H * e), P["o"])


def route(z, correction, groups, keep, top, scale):
    """Router logits of one token -> (chosen experts, their weights).  Choices are made on sigmoid + correction, among the
    experts of the groups whose two best choice scores sum up highest; weights are the plain sigmoids times scale."""
    s = sigmoid(z)
    choice = s + correction
    per = len(z) // groups
    score = [np.sort(choice[g * per:(g + 1) * per])[-2:].sum() for g in range(groups)]
    allowed = np.repeat(np.isin(np.arange(groups), np.argsort(-np.array(score), kind="stable")[:keep]), per)
    ids = np.argsort(-np.where(allowed, choice, -np.inf), kind="stable")[:top]
    return ids, s[ids] * scale


def moe_mlp(h, P, mlp):
    r, e, out = mlp["router"], mlp["expert"], np.zeros_like(h)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = linear(h, P["router"])
    for t in range(h.shape[0]):
        ids, w = route(z[t], P["correction"].reshape(-1), groups["count"], groups["keep"], r["top"], r["scale"])
        for i, wi in zip(ids, w):
            out[t] += wi * clamped_mlp(h[t:t + 1], {n: P[f"e{i}.{n}"] for n in ("gate", "up", "down")}, e["limit"])[0]
    return out


def mix_general_delta(h, P, m, eps, st):
    """S <- diag(w) S - (a u)(u^T S) + k v^T with the unit key u, o = S^T r; both terms read the old state."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    r, k, v = (linear(h, P[n]).reshape(T, H, d) for n in "rkv")
    w = decay_below_one(linear(np.tanh(linear(h, P["w1"])), P["w2"]) + P["w0"].reshape(-1)).reshape(T, H, d)
    a = sigmoid(linear(h, P["a"]) + P["a.b"].reshape(-1)).reshape(T, H, d)
    if "S" not in st:
        st["S"] = np.zeros((H, d, d), F)
    o = removal_rule(r, k, v, w, a, unit_vectors(k), st["S"])
    o = rms_norm(o, 1.0, eps).reshape(T, H * d) * P["norm"].reshape(-1)
    return linear(o * sigmoid(linear(h, P["g"])), P["o"])


def decay_below_one(z):
    """exp(-e^(-1/2) sigmoid(z)): between 0.545 and 1."""
    return np.exp(-np.exp(-0.5) * sigmoid(z))


def removal_rule(r, k, v, w, a, u, S):
    """All [T, H, d]; S [H, d, d] (changed in place).  Returns o [T, H, d]."""
    o = np.zeros_like(v)
    for t in range(r.shape[0]):
        for h in range(r.shape[1]):
            old = S[h].copy()
            S[h] = w[t, h][:, None] * old - np.outer(a[t, h] * u[t, h], u[t, h] @ old) + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ r[t, h]
    return o


def sigmoid_attention(q, k, v, pos, scale, bias, window=None):
    """q [T, H, d], k [n, G, d], v [n, G, e]: every visible key counts sigmoid(score + bias of the head), unnormalized."""
    T, H, _ = q.shape
    of = np.arange(H) // (H // k.shape[1])
    out = np.zeros((T, H, v.shape[2]), F)
    for t in range(T):
        n = int(pos[t]) + 1
        lo = max(0, n - window) if window else 0
        s = np.einsum("hd,nhd->hn", q[t], k[lo:n, of]) * scale + bias[:, None]
        out[t] = np.einsum("hn,nhe->he", sigmoid(s), v[lo:n, of])
    return out


def mix_sigmoid_attention(h, P, m, eps, pos, st):
    """Grouped-query attention without rotation: short convolutions, norms of queries, keys and values per head, sigmoid weights,
    a gate per head."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    z = {}
    for n in "qkv":
        z[n], st["conv." + n] = short_conv(linear(h, P[n]), P[n + ".conv"], None, st.get("conv." + n))
    q = rms_norm(z["q"].reshape(T, H, d), 1.0, eps)
    k, v = grow(st, k=rms_norm(z["k"].reshape(T, G, d), 1.0, eps), v=rms_norm(z["v"].reshape(T, G, e), 1.0, eps))
    o = sigmoid_attention(q, k, v, pos, m["scale"], P["pb"].reshape(-1), (m.get("mask") or {}).get("size"))
    o = o * sigmoid(linear(h, P["g"]))[:, :, None]
    return linear(o.reshape(T, H * e), P["o"])


def silu_mlp(h, P):
    return linear(silu(linear(h, P["gate"])) * linear(h, P["up"]), P["down"])


def softmax_route(z, top):
    """Router logits of one token -> (chosen experts, their weights): the largest softmax scores, divided by their sum."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    ids = np.argsort(-s, kind="stable")[:top]
    return ids, s[ids] / (s[ids].sum() + 1e-20)


def squared_relu_mlp(h, P):
    return linear(np.maximum(linear(h, P["up"]), 0.0) ** 2, P["down"])


def softmax_moe_mlp(h, P, mlp):
    out, z = np.zeros_like(h), linear(h, P["router"])
    for t in range(h.shape[0]):
        for i, wi in zip(*softmax_route(z[t], mlp["router"]["top"])):
            out[t] += wi * squared_relu_mlp(h[t:t + 1], {n: P[f"e{i}.{n}"] for n in ("up", "down")})[0]
    return out


def hyper_input(x, hc):
    """x [streams, T, W] -> the sublayer's input."""
    return np.einsum("s,stw->tw", hc["in"].reshape(-1), x)


def hyper_update(x, y, hc, mul):
    """Every stream anew from all old ones (mix: [from, to]) and the sublayer's output."""
    return np.einsum("st,snw->tnw", hc["mix"], x) + mul * hc["out"].reshape(-1)[:, None, None] * y


# ---------------------------------------------------------------- the decoder
def layer_runs(config):
    """(layer, pass that starts here or None) in the order in which layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    again = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + again + [(i, None) for i in range(b, n)]


class Stepper:
    def __init__(self, config: dict, tensors: dict):
        self.c = config
        self.w = {k: np.asarray(v, F) for k, v in tensors.items()}
        self.pos = 0
        self.runs = layer_runs(config)
        self.state = [dict() for _ in self.runs]

    def part(self, prefix):
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def step(self, tokens, trace=None):
        """Runs the next tokens of the sequence; returns their logits [n, vocab].  trace (a list) receives the
        residual after every layer."""
        tokens = np.asarray(tokens)
        pos = self.pos + np.arange(tokens.size)
        layer = {"Garilix": self.garilix_layer, "Datasun": self.datasun_layer, "Gomuzen": self.gomuzen_layer,
                 "Vepitar": self.vepitar_layer}[self.c["architecture"]]
        x = self.w["embed"][tokens] * self.c.get("embedding", {}).get("scale", 1.0)
        streams = self.c.get("streams")
        plus = 1.0 if streams else 0.0          # norm weights stored around zero
        if streams:
            x = np.stack([x] * streams)
        for st, (i, t) in zip(self.state, self.runs):
            if t is not None:
                x = x + self.w["loop.step"][t]
            x = layer(i, x, pos, st)
            if trace is not None:
                trace.append(x.sum(axis=0) if streams else x.copy())
        self.pos += tokens.size
        if streams:
            x = x.sum(axis=0)
        return linear(rms_norm(x, self.w["final.norm"] + plus, self.c["norm"]["eps"]), self.w["head" if "head" in self.w else "embed"])

    def garilix_layer(self, i, x, pos, st):
        L, P, eps = self.c["layers"][i], self.part(f"l{i}.mix."), self.c["norm"]["eps"]
        m = L["mixer"]
        if L["type"] == "channel_delta":
            y = mix_channel_delta(x, P, m, eps, st)
        elif L["type"] == "mamba2":
            y = mix_mamba2(x, P, m, eps, st)
        elif L["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                latent_append(x, P, m, eps, pos, st)
            y = mix_latent_attention(x, P, m, eps, pos, st if src is None else self.state[src])
        else:
            raise ValueError(L["type"])
        x = x + rms_norm(y, self.w[f"l{i}.norm1"], eps)
        if L.get("mlp"):
            x = x + rms_norm(dense_mlp(x, self.part(f"l{i}.mlp.")), self.w[f"l{i}.norm2"], eps)
        return x

    def datasun_layer(self, i, x, pos, st):
        L, P, eps = self.c["layers"][i], self.part(f"l{i}.mix."), self.c["norm"]["eps"]
        h = rms_norm(x, self.w[f"l{i}.norm1"], eps)
        if L["type"] == "attention":
            y = mix_attention(h, P, L["mixer"], eps, pos, st)
        elif L["type"] == "lightning":
            y = mix_lightning(h, P, L["mixer"], eps, st)
        else:
            raise ValueError(L["type"])
        if L.get("mlp"):
            y = y + clamped_mlp(h, self.part(f"l{i}.mlp."), L["mlp"]["limit"])
        return x + y

    def gomuzen_layer(self, i, x, pos, st):
        L, P, eps = self.c["layers"][i], self.part(f"l{i}.mix."), self.c["norm"]["eps"]
        h = rms_norm(x, self.w[f"l{i}.norm1"], eps)
        if L["type"] == "latent_attention":
            latent_append(h, P, L["mixer"], eps, pos, st)
            x = x + mix_latent_attention(h, P, L["mixer"], eps, pos, st)
        elif L["type"] == "attention":
            x = x + mix_differential(h, P, L["mixer"], eps, pos, st)
        elif L["type"] == "attention_2":
            x = x + mix_kept_window(h, P, L["mixer"], eps, pos, st)
        else:
            raise ValueError(L["type"])
        if L.get("mlp"):
            x = x + moe_mlp(rms_norm(x, self.w[f"l{i}.norm2"], eps), self.part(f"l{i}.mlp."), L["mlp"])
        return x

    def vepitar_layer(self, i, x, pos, st):
        L, P, eps, mul = self.c["layers"][i], self.part(f"l{i}.mix."), self.c["norm"]["eps"], self.c["residual_mult"]
        hc = self.part(f"l{i}.hc1.")
        h = rms_norm(hyper_input(x, hc), 1.0 + self.w[f"l{i}.norm1"], eps)
        if L["type"] == "general_delta":
            y = mix_general_delta(h, P, L["mixer"], eps, st)
        elif L["type"] == "attention":
            y = mix_sigmoid_attention(h, P, L["mixer"], eps, pos, st)
        else:
            raise ValueError(L["type"])
        x = hyper_update(x, y, hc, mul)
        if L.get("mlp"):
            hc, P = self.part(f"l{i}.hc2."), self.part(f"l{i}.mlp.")
            h = rms_norm(hyper_input(x, hc), 1.0 + self.w[f"l{i}.norm2"], eps)
            x = hyper_update(x, softmax_moe_mlp(h, P, L["mlp"]) if L["mlp"]["kind"] == "moe" else silu_mlp(h, P), hc, mul)
        return x


def forward(config, tensors, tokens):
    """(logits [T, vocab], residual after every layer run [runs, T, width]) of one whole sequence."""
    tr = []
    lg = Stepper(config, tensors).step(tokens, tr)
    return lg, np.stack(tr)


def greedy(config, tensors, prompt, n):
    s = Stepper(config, tensors)
    out = [int(np.argmax(s.step(prompt)[-1]))]
    while len(out) < n:
        out.append(int(np.argmax(s.step([out[-1]])[-1])))
    return out
