"""A plain, slow statement of the Lirutar decoder in NumPy: whole sequences, no cache, one function per mechanism.

It shares nothing with the engine: its own reader of config.json and model.safetensors, its own arithmetic (float64, so that it is the
sharper side of every comparison).

Notation.  T tokens of one sequence at positions 0..T-1; W the width; eps = norm.eps; LN(x; w, b) = (x - mean) / sqrt(var + eps) w + b.

    x0 = LN(E[id])                                   the embedding, normed
    every pass over the looped layers begins with    x <- W_in [x | x0]
    a layer:                                         x += mixer(LN1(x)),  then (unless null)  x += ff(LN2(x))
    logits = head LN(x)

  mixer         s_l attention(h) + s_r ssd(h), the two side by side on the same h
  attention     q, k, v with biases; the first `dims` values of every query and key head turned in pairs (i, i + dims/2) by p f_i,
                f_i = base^(-2i/dims); softmax(scale q.k) over the last `size` positions; W_o
  ssd           [z | x | B | C | dt] = W_in h;  (x, B, C) <- silu(causal convolution per channel + bias);  dt <- softplus(dt + b);
                per head S_t = e^(-e^A dt) S_(t-1) + dt B_t x_t^T,  y_t = S_t^T C_t + D x_t;  y silu(z), divided by its root mean
                square in norm_groups equal parts, times w;  W_o
  feed-forward  dense: W_d relu(W_u h)^2;  experts: p = softmax(W_r h) over experts and identities; the `top` largest p + c inside the
                `keep` groups with the largest maxima of p + c; weights p / (sum + 1e-20) times the router's scale; an identity gives h,
                an expert W_d (g sigmoid(1.702 g) (u + 1)), g = min(W_g h, L), u = clamp(W_u h, -L, L); plus the shared expert
"""
from __future__ import annotations

import json
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


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_parts(x, parts, eps):
    """Every one of `parts` equal parts of the last axis divided by its own root mean square."""
    y = x.reshape(*x.shape[:-1], parts, x.shape[-1] // parts)
    return (y / np.sqrt(np.mean(y * y, axis=-1, keepdims=True) + eps)).reshape(x.shape)


def layer_norm(x, w, b, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def turn_halves(x, pos, base, dims):
    """x [heads, T, n]: pairs (i, i + dims/2) of the first `dims` values turned by pos * base^(-2i/dims)."""
    half = dims // 2
    ang = np.asarray(pos, dtype=np.float64)[:, None] * (base ** (-2.0 * np.arange(half) / max(dims, 1)))[None, :]
    c, s = np.cos(ang), np.sin(ang)
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def attention(w, p, m, h):
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = np.arange(T)
    q, k, v = ((h @ w[p + n].T + w[p + n + ".b"]).reshape(T, heads, d).transpose(1, 0, 2) for n, heads, d in (("q", H, dk), ("k", G, dk), ("v", G, dv)))
    if m.get("rot") is not None:
        q, k = (turn_halves(t, pos, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
    back = pos[:, None] - pos[None, :]
    seen = back >= 0
    if m.get("mask") is not None:
        seen &= back < m["mask"]["size"]
    o = np.zeros((T, H, dv))
    for i in range(H):
        z = np.where(seen, q[i] @ k[i // (H // G)].T * m["scale"], -np.inf)
        e = np.exp(z - z.max(axis=1, keepdims=True))
        o[:, i] = (e / e.sum(axis=1, keepdims=True)) @ v[i // (H // G)]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n], the last column the current token's."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return sum(padded[j:j + len(x)] * taps[:, j] for j in range(n)) + bias


def ssd(w, p, m, h, eps):
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    T, inner = h.shape[0], H * dv
    row = h @ w[p + "in"].T
    z, xbc, dt = row[:, :inner], row[:, inner:2 * inner + 2 * G * N], row[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = xbc[:, :inner].reshape(T, H, dv), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    decay = np.exp(-np.exp(w[p + "A_log"]) * dt)
    S = np.zeros((H, N, dv))
    y = np.zeros((T, H, dv))
    for t in range(T):
        for i in range(H):
            g = i // (H // G)
            S[i] = decay[t, i] * S[i] + dt[t, i] * B[t, g][:, None] * x[t, i][None, :]
            y[t, i] = S[i].T @ C[t, g] + w[p + "D"][i] * x[t, i]
    y = y.reshape(T, inner) * silu(z)
    return (rms_parts(y, m["norm_groups"], eps) * w[p + "norm"]) @ w[p + "o"].T


def mixer(w, p, m, h, eps):
    return m["left_scale"] * attention(w, p + "left.", m["left"], h) + m["right_scale"] * ssd(w, p + "right.", m["right"], h, eps)


def expert(w, p, L, h):
    g = np.minimum(h @ w[p + "gate"].T, L)
    u = np.clip(h @ w[p + "up"].T, -L, L)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(z, correction, r):
    """One token's logits [experts + identities] -> [(index, weight)]."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    choice = s + correction
    count, keep = (r["groups"]["count"], r["groups"]["keep"]) if r.get("groups") else (1, 1)
    size = len(z) // count
    best = sorted(range(count), key=lambda g: -choice[g * size:(g + 1) * size].max())[:keep]
    allowed = [e for g in best for e in range(g * size, (g + 1) * size)]
    chosen = sorted(allowed, key=lambda e: -choice[e])[:r["top"]]
    total = sum(s[e] for e in chosen) + 1e-20
    return [(e, s[e] / total * r.get("scale", 1.0)) for e in chosen]


def experts_ff(w, p, mlp, h):
    r = mlp["router"]
    z = h @ w[p + "router"].T
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in route(z[t], w[p + "correction"], r):
            out[t] += weight * (h[t] if e >= r["experts"] else expert(w, f"{p}e{e}.", mlp["expert"]["limit"], h[t:t + 1])[0])
    if mlp.get("shared") is not None:
        out += expert(w, p + "shared.", mlp["shared"]["limit"], h)
    return out


def dense_ff(w, p, h):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def runs(cfg):
    """[(layer, whether it begins a pass over the looped layers)] in the order they run."""
    n = len(cfg["layers"])
    if cfg.get("loop") is None:
        return [(i, False) for i in range(n)]
    a, b, times = (cfg["loop"][k] for k in ("start", "stop", "times"))
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(times) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def forward(cfg, w, ids, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the residual stream after every run of a layer."""
    eps = cfg["norm"]["eps"]
    n = lambda name, v: layer_norm(v, w[name], w[name + ".b"], eps)
    x0 = n("embed.norm", w["embed"][np.asarray(ids, dtype=np.int64)])
    x = x0
    for i, begins in runs(cfg):
        if begins:
            x = np.concatenate([x, x0], axis=1) @ w["loop.in"].T
        layer = cfg["layers"][i]
        x = x + mixer(w, f"l{i}.mix.", layer["mixer"], n(f"l{i}.norm1", x), eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = n(f"l{i}.norm2", x)
            x = x + (dense_ff(w, f"l{i}.mlp.", h) if mlp["kind"] == "dense" else experts_ff(w, f"l{i}.mlp.", mlp, h))
        if layers_out is not None:
            layers_out.append(x.copy())
    return n("final.norm", x) @ w["head"].T
