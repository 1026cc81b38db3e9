"""A plain, slow statement of the Dubazen design in torch on the CPU: one function per mechanism, whole sequences at a
time, recurrences token by token, no cache.  It shares no code with the engine; the tests compare the engine with it.

``cfg`` is the parsed ``config.json`` (a dict), ``W`` maps tensor names to tensors of the working precision
(float32, or float64 for a sharper oracle).
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


# --------------------------------------------------------------------------- small pieces
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def scalar_rms_norm(x, g, eps):
    return rms(x, eps) * g.reshape(())


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def turn_halves(x, dims, base, sign=1.0):
    """x [n, heads, d]: pair i < dims/2 is (x_i, x_{i + dims/2}), turned by sign * position * base^(-2i/dims);
    positions are the rows' indices; elements from ``dims`` on pass unchanged."""
    n, half = x.shape[0], dims // 2
    out = x.clone()
    pos = torch.arange(n, dtype=torch.float32)
    for i in range(half):
        ang = pos * torch.tensor(float(base) ** (-2.0 * i / dims), dtype=torch.float32)    # 32-bit angles
        c, s = torch.cos(ang).to(x.dtype)[:, None], sign * torch.sin(ang).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def causal_conv(x, w, b):
    """x [n, C], w [C, taps] with the last column the current token's, zeros before the start."""
    n, C = x.shape
    taps = w.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, C), x])
    y = b.expand(n, C).clone()
    for j in range(taps):
        y = y + padded[j:j + n] * w[:, j]
    return y


# --------------------------------------------------------------------------- mixers
def softmax_with_sink(scores, sink):
    """[n, n] causal weights: exp(score) over exp(sink) plus the sum of exp(score) of the keys up to the query's."""
    n = scores.shape[0]
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    s = torch.where(j <= i, scores, torch.full_like(scores, -math.inf))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def turned_value_attention(h, W, p, m, eps):
    """Attention whose queries and keys are rotated, then divided by their root mean square; values are turned with
    their position and a head's result turned back with the query's; sinks; output gate; biases."""
    n = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, V = m.get("kv_heads", H), m.get("vdim", D)
    q = _r(h @ W[p + "q"].T + W[p + "q.b"]).view(n, H, D)
    k = _r(h @ W[p + "k"].T + W[p + "k.b"]).view(n, G, D)
    v = _r(h @ W[p + "v"].T + W[p + "v.b"]).view(n, G, V)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q = _r(rms(turn_halves(q, dims, base), eps))
    k = _r(rms(turn_halves(k, dims, base), eps))
    v = _r(turn_halves(v, V, base))
    o = torch.zeros(n, H, V, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        w = softmax_with_sink(q[:, a] @ k[:, g].T * m["scale"], W[p + "sink"][a])
        o[:, a] = _r(w) @ v[:, g]
    o = turn_halves(o, V, base, -1.0)
    y = o.reshape(n, H * V) * torch.sigmoid(_r(h @ W[p + "g"].T))
    return _r(y) @ W[p + "o"].T + W[p + "o.b"]


def fixed_decay_attention(h, W, p, m, eps):
    """S <- d S + k v^T, o = S^T q on SiLU(q, k, v), one fixed decay a head."""
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m.get("vdim", m["dim"])
    q = silu(_r(h @ W[p + "q"].T)).view(n, H, D)
    k = silu(_r(h @ W[p + "k"].T)).view(n, H, D)
    v = silu(_r(h @ W[p + "v"].T)).view(n, H, V)
    d = torch.tensor([float(x) for x in m["decay"]], dtype=h.dtype)[:, None, None]
    S = h.new_zeros(H, D, V)
    out = h.new_zeros(n, H, V)
    for t in range(n):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    o = rms(out.reshape(n, H * V), eps) * W[p + "norm"]
    return _r(o * torch.sigmoid(_r(h @ W[p + "g"].T))) @ W[p + "o"].T


def parallel(h, W, p, m, eps):
    return (m["left_scale"] * turned_value_attention(h, W, p + "left.", m["left"], eps)
            + m["right_scale"] * fixed_decay_attention(h, W, p + "right.", m["right"], eps))


def gated_linear_attention(h, W, p, m, eps):
    """S <- diag(alpha) S + k v^T, o = S^T q; alpha = sigmoid(A2 (A1 h) + b)^(1/tau) per key channel."""
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m.get("vdim", m["dim"])
    q = (_r(h @ W[p + "q"].T) * D ** -0.5).view(n, H, D)
    k = _r(h @ W[p + "k"].T).view(n, H, D)
    v = _r(h @ W[p + "v"].T).view(n, H, V)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / m["tau"])).view(n, H, D)
    S = h.new_zeros(H, D, V)
    out = h.new_zeros(n, H, V)
    for t in range(n):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    o = (rms(out, eps) * W[p + "norm"]).reshape(n, H * V)
    return _r(o * silu(_r(h @ W[p + "g"].T))) @ W[p + "o"].T


def selective_scan(h, W, p, m, eps):
    """A channel's state row decays by e^(-step e^A_log), gains step x B and is read by C; D x beside it, a gate behind."""
    n, I, N, R = h.shape[0], m["inner"], m["state"], m["dt_rank"]
    xz = _r(h @ W[p + "in"].T)
    x, z = xz[:, :I], xz[:, I:]
    x = _r(silu(causal_conv(x, W[p + "conv"], W[p + "conv.b"])))
    low = x @ W[p + "x"].T
    dt, B, C = low[:, :R], low[:, R:R + N], low[:, R + N:]
    dt = softplus(dt @ W[p + "dt"].T + W[p + "dt.b"])
    A = -torch.exp(W[p + "A_log"])
    S = h.new_zeros(I, N)
    y = h.new_zeros(n, I)
    for t in range(n):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = (S * C[t][None, :]).sum(1) + W[p + "D"] * x[t]
    return _r(y * silu(z)) @ W[p + "o"].T


MIXERS = {"parallel": parallel, "gla": gated_linear_attention, "mamba1": selective_scan}


# --------------------------------------------------------------------------- feed-forward
def expert(W, p, h, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, min=-limit, max=limit)
    return _r(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def experts(f, W, p, h):
    """The ``top`` largest softmax scores, divided by their sum, weigh their experts; a shared expert is added."""
    top = f["router"]["top"]
    s = torch.softmax(h @ W[p + "router"].T, dim=-1)
    w, ids = torch.topk(s, top, dim=-1)
    w = w / (w.sum(-1, keepdim=True) + 1e-20)
    y = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, j = torch.where(ids == e)
        if t.numel():
            y[t] += w[t, j][:, None] * expert(W, f"{p}e{e}.", h[t], f["expert"]["limit"])
    if f.get("shared") is not None:
        y = y + expert(W, p + "shared.", h, f["shared"]["limit"])
    return y


# --------------------------------------------------------------------------- the model
def mix_streams(X, y, mix, out):
    """X [streams, n, width]: new X_t = sum_s mix[s, t] X_s + out[t] y."""
    return torch.einsum("snw,st->tnw", X, mix) + out[:, None, None] * y[None]


def read_streams(X, weights):
    return torch.einsum("snw,s->nw", X, weights)


def forward(cfg, W, tokens, return_layers=False):
    """[n, vocab] logits of a whole sequence (and the sum of the streams after every layer)."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    X = x[None].repeat(cfg["streams"], 1, 1)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        u = _r(scalar_rms_norm(read_streams(X, W[p + "hc1.in"]), W[p + "norm1"], eps))
        X = mix_streams(X, MIXERS[layer["type"]](u, W, p + "mix.", layer["mixer"], eps), W[p + "hc1.mix"], W[p + "hc1.out"])
        if layer.get("mlp") is not None:
            u = _r(scalar_rms_norm(read_streams(X, W[p + "hc2.in"]), W[p + "norm2"], eps))
            X = mix_streams(X, experts(layer["mlp"], W, p + "mlp.", u), W[p + "hc2.mix"], W[p + "hc2.out"])
        after.append(X.sum(0))
    logits = _r(scalar_rms_norm(X.sum(0), W["final.norm"], eps)) @ W["head"].T
    return (logits, after) if return_layers else logits


def greedy(cfg, W, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):]


def load_weights(folder, dtype=torch.float32):
    """The tensors of a model folder, read here byte by byte, in the working precision."""
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
        else:
            assert info["dtype"] == "F32", info["dtype"]
            t = torch.from_numpy(raw.view(np.float32)).to(dtype)
        out[name] = t.reshape(info["shape"])
    return out
