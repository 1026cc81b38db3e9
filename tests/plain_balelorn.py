"""A plain, slow statement of the Balelorn design in torch on the CPU: one function per mechanism, whole sequences at
a time, no cache.  It shares no code with the engine; the tests compare the engine with it.

``cfg`` is the parsed ``config.json`` (a dict), ``W`` maps tensor names to tensors of the working precision
(float32, or float64 for a sharper oracle; integer tables as integers).
"""
from __future__ import annotations

import contextlib
import math

import torch

_ROUND = None      # an element type that everything the design allows in 16 bits is rounded to (None: nothing is)


@contextlib.contextmanager
def rounded_to(dtype):
    """Inside: what an engine may keep in ``dtype`` (the products' inputs and outputs) is rounded to it, so that the
    distance to the unrounded result shows what rounding alone does."""
    global _ROUND
    old, _ROUND = _ROUND, dtype
    try:
        yield
    finally:
        _ROUND = old


def _r(x):
    return x.to(_ROUND).to(x.dtype) if _ROUND is not None else x


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def rotate_halves(x, dims, base):
    """x [n, heads, d]: pair i < dims/2 is (x_i, x_{i + dims/2}), turned by position * base^(-2i/dims); positions are
    the rows' indices; elements from ``dims`` on pass unchanged."""
    n, half = x.shape[0], dims // 2
    out = x.clone()
    pos = torch.arange(n, dtype=torch.float32)
    for i in range(half):
        ang = pos * torch.tensor(float(base) ** (-2.0 * i / dims), dtype=torch.float32)    # 32-bit angles
        c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def chunk_mask(n, size):
    """[n, n]: query i sees key j if j <= i and both lie in the same chunk of ``size`` positions (None: one chunk)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    m = j <= i
    if size is not None:
        m = m & (i // size == j // size)
    return m


def softmax_with_sink(scores, mask, sink):
    """[n, n] weights: exp(score) over exp(sink) plus the sum of exp(score) of the visible keys."""
    s = torch.where(mask, scores, torch.full_like(scores, -math.inf))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def mixed_values(v, first, lam):
    """(1 - lambda) v + lambda first."""
    return (1.0 - lam) * v + lam * first


def attention(m, W, p, h, first):
    """Returns (output before the block's norm, the layer's values as projected).  ``first``: the values of the first
    layer that takes part in the mixing of values (None: this layer is that one, or takes no part)."""
    n = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, V = m.get("kv_heads", H), m.get("vdim", D)
    q = _r(h @ W[p + "q"].T).view(n, H, D)
    k = _r(h @ W[p + "k"].T).view(n, G, D)
    v = _r(h @ W[p + "v"].T).view(n, G, V)
    projected = v
    rot = m.get("rot")
    if rot and rot.get("dims"):
        q, k = rotate_halves(q, rot["dims"], rot["base"]), rotate_halves(k, rot["dims"], rot["base"])
    if first is not None:
        v = mixed_values(v, first.reshape(v.shape), W[p + "vmix"])    # (element by element of the rows [kv head][vdim])
    q, k, v = _r(q), _r(k), _r(v)
    mask = chunk_mask(n, m["mask"]["size"] if m.get("mask") else None)
    o = torch.zeros(n, H, V, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        w = softmax_with_sink(q[:, a] @ k[:, g].T * m["scale"], mask, W[p + "sink"][a])
        o[:, a] = _r(w) @ v[:, g]
    y = o.reshape(n, H * V) * torch.sigmoid(_r(h @ W[p + "g"].T))
    return _r(y) @ W[p + "o"].T, projected


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def dense(f, W, p, h):
    return _r(gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert(W, p, h, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, min=-limit, max=limit)
    return _r(_r(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T)


def table_experts(f, W, p, h, tokens):
    """Each token's experts are the entries of its row of the table, with equal weights."""
    top = f["router"]["top"]
    y = torch.zeros_like(h)
    table = W[p + "table"]
    for t, tok in enumerate(tokens):
        for j in range(top):
            e = int(table[tok, j])
            y[t] += expert(W, f"{p}e{e}.", h[t:t + 1], f["expert"]["limit"])[0] / top
    return y


def feed_forward(f, W, p, h, tokens):
    if f["kind"] == "dense":
        return dense(f, W, p, h)
    assert f["kind"] == "moe"
    return table_experts(f, W, p, h, tokens)


def forward(cfg, W, tokens, return_layers=False):
    """[n, vocab] logits of a whole sequence (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    x = rms_norm(W["embed"][torch.tensor(tokens)], W["embed.norm"], eps)
    first, after = None, []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m, f = layer["mixer"], layer.get("mlp")
        mixes = bool(m.get("v_mix"))
        y, values = attention(m, W, p + "mix.", _r(rms_norm(x, W[p + "norm1"], eps)), first if mixes else None)
        if mixes and first is None:
            first = values
        x = x + rms_norm(y, W[p + "norm1b"], eps) * W[p + "ls1"]
        if f is not None:
            y = feed_forward(f, W, p + "mlp.", _r(rms_norm(x, W[p + "norm2"], eps)), tokens)
            x = x + rms_norm(y, W[p + "norm2b"], eps) * W[p + "ls2"]
        after.append(x)
    logits = _r(rms_norm(x, W["final.norm"], eps)) @ W["head"].T
    return (logits, after) if return_layers else logits


def greedy(cfg, W, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):]


def load_weights(folder, dtype=torch.float32):
    """The tensors of a model folder, read here byte by byte, in the working precision (integers as int64)."""
    import json
    import os
    import struct

    import numpy as np

    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        raw = np.frombuffer(data[a:b], dtype=np.uint8).copy()
        if info["dtype"] == "BF16":
            t = torch.from_numpy((raw.view(np.uint16).astype(np.uint32) << 16).view(np.float32)).to(dtype)
        elif info["dtype"] == "F32":
            t = torch.from_numpy(raw.view(np.float32)).to(dtype)
        else:
            assert info["dtype"] == "I32", info["dtype"]
            t = torch.from_numpy(raw.view(np.int32)).to(torch.int64)
        out[name] = t.reshape(info["shape"])
    return out
