"""Small Lirutar models for the tests: configurations of the tests' own, random weights of the tests' own making.

None of the configurations is anybody's model.  Between them they vary what a single model would make equal or 1: query against
key-value heads, key against value sizes, fewer turned values than a head has, all of them or none, windows of one, shorter and longer
than a page, a chunk of the recurrence and a prompt, or none; heads a group of the state-space mixer, state rows against values, taps,
parts of its norm, the two scales; experts with and without identities, groups, a correction that reverses the choice, a shared expert,
a router scale of 1 and others; layers without a feed-forward; loops over the first layers, over inner ones, over all, once, three times
and none; sizes the tensor-core kernels take and sizes they refuse.
"""
import json
import os

import numpy as np
import torch


def att(heads, kv, dim, vdim, scale, rot=None, window=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale)
    if rot is not None:
        m["rot"] = dict(base=rot[0], dims=rot[1])
    if window is not None:
        m["mask"] = dict(size=window)
    return m


def ssd(heads, vdim, state, groups, conv, norm_groups):
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, limit, experts, top, identity=0, count=1, keep=1, scale=1.0, shared=None):
    d = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top, identity=identity, scale=scale,
                                                                      groups=dict(count=count, keep=keep)))
    if shared is not None:
        d["shared"] = dict(ff=shared[0], limit=shared[1])
    return d


def layer(left, right, mlp=None, left_scale=1.0, right_scale=1.0):
    return dict(type="parallel", mixer=dict(left=left, right=right, left_scale=left_scale, right_scale=right_scale), mlp=mlp)


def config(vocab, width, layers, loop=None, eps=1e-5):
    d = dict(architecture="Lirutar", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# every kind of feed-forward and none; inner layers looped three times; windows shorter and longer than a page of eight
CFG_ALL = config(97, 64, [layer(att(4, 2, 16, 24, 0.3, (10000.0, 8), 21), ssd(4, 12, 20, 2, 4, 2), dense(96), 0.7, 1.3),
                          layer(att(2, 1, 24, 8, 0.25, (300.0, 24), 5), ssd(2, 24, 16, 1, 3, 1), moe(24, 1.2, 6, 2, 2, 4, 2, 1.7, (40, 0.8)), 1.1, 0.4),
                          layer(att(3, 3, 8, 16, 0.5, None, 70), ssd(6, 8, 32, 3, 2, 3), None, 0.5, 0.9),
                          layer(att(4, 1, 16, 16, 0.35, (50.0, 4)), ssd(3, 16, 24, 3, 4, 1), moe(16, 0.7, 5, 3), 1.0, 1.0)],
                 loop=(1, 3, 3))
# odd sizes that only the general kernels take; all layers looped once; a window of one; one tap
CFG_ODD = config(61, 40, [layer(att(3, 1, 10, 14, 0.4, (50.0, 6), 1), ssd(3, 7, 5, 1, 1, 7), moe(12, 2.0, 3, 2, 3, 2, 1, 0.6, (20, 1.5)), 0.9, 0.6),
                          layer(att(5, 5, 6, 10, 0.6, (7.0, 2), 33), ssd(5, 9, 11, 5, 5, 1), dense(56), 1.4, 0.3)],
                 loop=(0, 2, 1), eps=1e-6)
# tensor-core sizes: wide heads, state rows and values of several chunks' worth, no loop at all
CFG_WIDE = config(83, 128, [layer(att(4, 1, 64, 128, 0.125, (200000.0, 32), 50), ssd(4, 64, 128, 2, 4, 4), moe(64, 1.25, 12, 3, 4, 4, 2, 2.5, (96, 1.0)), 0.8, 0.7),
                            layer(att(2, 2, 32, 96, 0.18, (1000.0, 32), 130), ssd(2, 80, 40, 1, 4, 8), dense(256), 0.6, 0.9)])
# the first layers looped twice, fewer layers behind
CFG_FRONT = config(71, 96, [layer(att(2, 1, 32, 32, 0.2, (5000.0, 16), 40), ssd(3, 32, 48, 3, 4, 3), dense(128), 0.7, 0.8),
                            layer(att(4, 4, 32, 64, 0.2, (5000.0, 16), 40), ssd(8, 16, 16, 2, 4, 2), moe(32, 1.0, 7, 2, 1, 2, 1, 1.2), 0.9, 0.5),
                            layer(att(2, 1, 32, 32, 0.2, (5000.0, 16), 40), ssd(3, 32, 48, 3, 4, 3), dense(128), 0.7, 0.8)],
                   loop=(0, 2, 2))

CONFIGS = {"all": CFG_ALL, "odd": CFG_ODD, "wide": CFG_WIDE, "front": CFG_FRONT}


def make_tensors(cfg, seed):
    """name -> float32 array, drawn so that every mechanism matters: biases and norm weights away from 0 and 1, scores of order one and
    more, step sizes and decays spread between fast and slow, clamps reached by a good part of the values, corrections as large as the
    differences of the scores (and of both signs), so that they move the choice but not the weights."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    n = lambda *shape, std=1.0: (rng.standard_normal(shape) * std).astype(np.float32)
    t = {"embed": n(V, W), "head": n(V, W, std=W ** -0.5)}

    def norm(name):
        t[name], t[name + ".b"] = 1 + n(W, std=0.2), n(W, std=0.15)

    def gated(p, ff):
        t[p + "gate"], t[p + "up"], t[p + "down"] = n(ff, W, std=1.5 * W ** -0.5), n(ff, W, std=1.5 * W ** -0.5), n(W, ff, std=ff ** -0.5)

    norm("embed.norm")
    norm("final.norm")
    if cfg.get("loop") is not None:
        t["loop.in"] = n(W, 2 * W, std=0.8 * W ** -0.5)
    for i, l in enumerate(cfg["layers"]):
        p, m, r = f"l{i}.", l["mixer"]["left"], l["mixer"]["right"]
        norm(p + "norm1")
        for name, rows, std in (("q", m["heads"] * m["dim"], 1.5), ("k", m["kv_heads"] * m["dim"], 1.5), ("v", m["kv_heads"] * m["vdim"], 1.5)):
            t[f"{p}mix.left.{name}"], t[f"{p}mix.left.{name}.b"] = n(rows, W, std=std * W ** -0.5), n(rows, std=0.5)
        t[p + "mix.left.o"] = n(W, m["heads"] * m["vdim"], std=(m["heads"] * m["vdim"]) ** -0.5)
        inner, chan, H = r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"], r["heads"]
        q = p + "mix.right."
        t[q + "in"] = n(inner + chan + H, W, std=1.3 * W ** -0.5)
        t[q + "conv"], t[q + "conv.b"] = n(chan, r["conv"], std=0.7), n(chan, std=0.2)
        t[q + "dt_bias"], t[q + "A_log"], t[q + "D"] = n(H, std=1.5) - 1.0, n(H, std=1.0), 1 + n(H, std=0.5)
        t[q + "norm"], t[q + "o"] = 1 + n(inner, std=0.2), n(W, inner, std=inner ** -0.5)
        ff = l["mlp"]
        if ff is None:
            continue
        norm(p + "norm2")
        if ff["kind"] == "dense":
            t[p + "mlp.up"], t[p + "mlp.down"] = n(ff["ff"], W, std=1.3 * W ** -0.5), n(W, ff["ff"], std=ff["ff"] ** -0.5)
        else:
            every = ff["router"]["experts"] + ff["router"].get("identity", 0)
            for e in range(ff["router"]["experts"]):
                gated(f"{p}mlp.e{e}.", ff["expert"]["ff"])
            t[p + "mlp.router"], t[p + "mlp.correction"] = n(every, W, std=2 * W ** -0.5), n(every, std=0.2)
            if ff.get("shared") is not None:
                gated(p + "mlp.shared.", ff["shared"]["ff"])
    return t


def write_model(model_dir, cfg, tensors, dtype=torch.bfloat16):
    """config.json and model.safetensors, stored in `dtype` (the values a bfloat16 checkpoint holds are what both the engine and the
    plain implementation then read)."""
    from vitna_anchor_b200.weights import write_model_folder
    os.makedirs(model_dir, exist_ok=True)
    write_model_folder(str(model_dir), cfg, {k: torch.from_numpy(np.ascontiguousarray(v)).to(dtype) for k, v in tensors.items()})
    with open(os.path.join(model_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    return str(model_dir)


def make_model(model_dir, name, seed=0):
    return write_model(model_dir, CONFIGS[name], make_tensors(CONFIGS[name], seed))
