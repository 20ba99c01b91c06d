"""Shared pieces of the layer-list decoders' tests: model folders, runs in portions, comparisons."""
from __future__ import annotations

import json
import os
import struct

import numpy as np

from oracle import layers_ref

TOL = {"float32": (2e-5, 5e-5), "bfloat16": (2.5e-2, 0.12)}      # median and largest relative error of a position


def close(got, want, dtype):
    e = rel(got, want)
    return np.median(e) < TOL[dtype][0] and e.max() < TOL[dtype][1]


def bf16_round(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def write_model(path, cfg, tensors, f32=()):
    """config.json and model.safetensors; tensors named in f32 are stored as F32, the others as BF16."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, off = {"__metadata__": {"note": "test"}}, [], 0
    for n, a in tensors.items():
        a = np.ascontiguousarray(a, dtype=np.float32)
        b = a.tobytes() if n in f32 else (a.view(np.uint32) >> 16).astype(np.uint16).tobytes()
        header[n] = {"dtype": "F32" if n in f32 else "BF16", "shape": list(a.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    h = json.dumps(header).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return str(path)


def rel(got, want):
    """Root mean square of the difference of each row over that of the wanted rows (means taken off)."""
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d ** 2).mean(axis=-1)) / np.sqrt((w ** 2).mean())


class ModelCase:
    """A model on disk, random tokens and their reference logits (of every position)."""

    def __init__(self, path, cfg, tensors, n=150, seed=0):
        self.cfg, self.tensors = cfg, tensors
        self.path = write_model(path, cfg, self.tensors)
        rng = np.random.default_rng(seed + 1)
        self.tokens = rng.integers(0, cfg["vocab"], size=n)
        self.want = layers_ref.Stepper(cfg, self.tensors).step(self.tokens)

    def model(self, ctx, dtype, max_seqs=4, max_ctx=512, pool_tokens=0, chunk=None):
        import densecore_b200 as dc
        m = dc.Model.from_dir(ctx, self.path, dtype, max_seqs, max_ctx, pool_tokens)
        if chunk:
            m.set_option("prefill_chunk", chunk)
        m.finalize()
        return m


def run(m, tokens, cuts):
    """One sequence in portions (cuts: their lengths, repeated as needed); logits of every position."""
    s, out, i, j = m.seq_alloc(), [], 0, 0
    while i < len(tokens):
        n = min(cuts[j % len(cuts)], len(tokens) - i)
        out.append(m.forward_batch([(s, tokens[i:i + n])], np.arange(n)))
        i, j = i + n, j + 1
    m.seq_free(s)
    return np.concatenate(out)
