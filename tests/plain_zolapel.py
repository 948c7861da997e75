"""A plain, slow statement of the Zolapel decoder in NumPy: whole sequences, no cache, one function per mechanism.

It shares nothing with the engine: its own reader of config.json and model.safetensors, its own arithmetic (float64, so that it is the
sharper side of every comparison).

Notation.  T tokens of one sequence at positions 0..T-1; W the width; eps = norm.eps; m = residual_mult; LN(x; w, b) = (x - mean) /
sqrt(var + eps) w + b; rms(x) = x / sqrt(mean(x^2) + eps).

    x0 = E[id]
    pass t over the looped layers begins with    x <- x (+ x0 if t > 0) + step_t
    layer i:    x += m ls1 attention(LN1(x));  x += m ls2 experts(LN2(x)) (unless null);
                y = P_i (gelu(G_i x) S[id, i-th part]);  x += m rms(y) n_i
    logits = E LN(x)

  attention     q, k = W_q h, W_k h; values are k as it is here; q, k <- rms per head, weighted; the first `dims` values of every query and
                key head turned in pairs (2i, 2i+1) by p f_i; softmax(scale q.k) over the last `size` positions; each head's output times
                sigmoid of its number of W_g h; W_o
  f_i           base^(-2i/dims), and with a scaling: divided by `factor` where the wavelength is above original/low, as it is below
                original/high, between the two a blend that is linear in original/wavelength
  experts       s = sigmoid(W_r h); the `top` largest; sum over them of W_d relu(W_u (s h))^2
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np


def read_tensors(path):
    """name -> float64 array."""
    with open(path, "rb") as f:
        raw = f.read()
    (n,) = struct.unpack("<Q", raw[:8])
    directory = json.loads(raw[8:8 + n].decode("utf-8"))
    out = {}
    for name, d in directory.items():
        if name == "__metadata__":
            continue
        lo, hi = d["data_offsets"]
        blob = raw[8 + n + lo:8 + n + hi]
        if d["dtype"] == "BF16":
            a = (np.frombuffer(blob, "<u2").astype(np.uint32) << 16).view("<f4").astype(np.float64)
        elif d["dtype"] == "F32":
            a = np.frombuffer(blob, "<f4").astype(np.float64)
        else:
            raise ValueError(f"{name}: dtype {d['dtype']}")
        out[name] = a.reshape(d["shape"])
    return out


def read_model(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_tensors(os.path.join(model_dir, "model.safetensors"))


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def frequencies(base, dims, scaling=None):
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            length = 2.0 * math.pi / f
            if length > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif length >= scaling["original"] / scaling["high"]:
                s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return np.array(out)


def turn_neighbours(x, pos, f):
    """x [heads, T, n]: pairs (2i, 2i+1) of the first 2 len(f) values turned by pos * f_i."""
    n = 2 * len(f)
    ang = np.asarray(pos, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(ang), np.sin(ang)
    out = x.copy()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


def attention(w, p, m, h, eps):
    H, d = m["heads"], m["dim"]
    G = m.get("kv_heads", H)
    T = h.shape[0]
    pos = np.arange(T)
    q = (h @ w[p + "q"].T).reshape(T, H, d).transpose(1, 0, 2)
    v = (h @ w[p + "k"].T).reshape(T, G, d).transpose(1, 0, 2)
    q, k = rms(q, eps) * w[p + "q.norm"], rms(v, eps) * w[p + "k.norm"]
    if m.get("rot") is not None:
        f = frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
        q, k = turn_neighbours(q, pos, f), turn_neighbours(k, pos, f)
    back = pos[:, None] - pos[None, :]
    seen = back >= 0
    if m.get("mask") is not None:
        seen &= back < m["mask"]["size"]
    gate = sigmoid(h @ w[p + "g"].T)
    o = np.zeros((T, H, d))
    for i in range(H):
        z = np.where(seen, q[i] @ k[i // (H // G)].T * m["scale"], -np.inf)
        e = np.exp(z - z.max(axis=1, keepdims=True))
        o[:, i] = gate[:, i:i + 1] * ((e / e.sum(axis=1, keepdims=True)) @ v[i // (H // G)])
    return o.reshape(T, H * d) @ w[p + "o"].T


def expert(w, p, h):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def experts_ff(w, p, mlp, h):
    s = sigmoid(h @ w[p + "router"].T)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in sorted(range(s.shape[1]), key=lambda e: -s[t, e])[:mlp["router"]["top"]]:
            out[t] += expert(w, f"{p}e{e}.", s[t, e] * h[t])
    return out


def side_input(w, p, x, e, eps):
    """What the token's own part e [T, dim] of the second table adds (before residual_mult)."""
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms(y, eps) * w[p + "norm"]


def runs(cfg):
    """[(layer, the number of the pass over the looped layers that begins with it, or -1)] in the order they run."""
    n = len(cfg["layers"])
    if cfg.get("loop") is None:
        return [(i, -1) for i in range(n)]
    a, b, times = (cfg["loop"][k] for k in ("start", "stop", "times"))
    return [(i, -1) for i in range(a)] + [(i, t if i == a else -1) for t in range(times) for i in range(a, b)] + [(i, -1) for i in range(b, n)]


def forward(cfg, w, ids, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the residual stream after every run of a layer."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    n = lambda name, v: layer_norm(v, w[name], w[name + ".b"], eps)
    ids = np.asarray(ids, dtype=np.int64)
    x0 = w["embed"][ids]
    x = x0
    for i, begins in runs(cfg):
        if begins > 0:
            x = x + x0
        if begins >= 0:
            x = x + w["loop.step"][begins]
        layer, p = cfg["layers"][i], f"l{i}."
        x = x + m * w[p + "ls1"] * attention(w, p + "mix.", layer["mixer"], n(p + "norm1", x), eps)
        if layer.get("mlp") is not None:
            x = x + m * w[p + "ls2"] * experts_ff(w, p + "mlp.", layer["mlp"], n(p + "norm2", x))
        if cfg.get("token_side") is not None:
            d = cfg["token_side"]["dim"]
            x = x + m * side_input(w, p + "side.", x, w["side.embed"][ids, i * d:(i + 1) * d], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return n("final.norm", x) @ w["embed"].T
