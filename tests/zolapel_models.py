"""Small Zolapel models for the tests: configurations of the tests' own, random weights of the tests' own making.

None of the configurations is anybody's model.  Between them they vary what a single model would make equal or 1: query against key heads,
fewer turned values than a head has, all of them or none, frequencies that are kept, divided and blended; windows of one, shorter and longer than a
page, a run of keys and a prompt, or none; one expert a token, several and all; layers without a feed-forward; models without the second table;
factors of 1 and others; loops over the first layers, over inner ones, over the last, once, three times and none; heads of sizes the tensor-core
kernels take and of sizes they refuse, an odd number of them.
"""
import json
import os

import numpy as np
import torch

BANDS = dict(factor=8.0, low=1.0, high=4.0, original=64)        # with these bases some frequencies are kept, some blended, some divided


def att(heads, kv, dim, scale, rot=None, window=None, scaling=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale)
    if rot is not None:
        m["rot"] = dict(base=rot[0], dims=rot[1])
        if scaling is not None:
            m["rot"]["scaling"] = dict(scaling)
    if window is not None:
        m["mask"] = dict(size=window)
    return m


def moe(ff, experts, top):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def layer(mixer, mlp=None):
    return dict(type="attention", mixer=mixer, mlp=mlp)


def config(vocab, width, layers, loop=None, side=None, mult=None, eps=1e-5):
    d = dict(architecture="Zolapel", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    if side is not None:
        d["token_side"] = dict(dim=side)
    if mult is not None:
        d["residual_mult"] = mult
    return d


# one expert a token, several, none; inner layers looped three times; windows shorter and longer than a page of eight
CFG_ALL = config(97, 64, [layer(att(4, 2, 16, 0.3, (10000.0, 8), 21, BANDS), moe(24, 6, 2)), layer(att(2, 1, 24, 0.25, (300.0, 24), 5), moe(40, 5, 1)),
                          layer(att(3, 3, 8, 0.5, None, 70), None), layer(att(4, 1, 32, 0.35, (50.0, 4)), moe(16, 4, 3))],
                 loop=(1, 3, 3), side=12, mult=0.6)
# sizes that only the general kernels take, an odd number of heads; the last layer looped once; a window of one; all experts; no second table
CFG_ODD = config(61, 42, [layer(att(3, 1, 10, 0.4, (50.0, 6), 1), moe(13, 3, 3)), layer(att(5, 5, 7, 0.6, (7.0, 2), 33), moe(20, 7, 2))], loop=(1, 2, 1), eps=1e-6,
                 mult=1.3)
# tensor-core sizes, prompts long enough for the grouped products, no loop, a factor of 1 by being left out
CFG_WIDE = config(83, 128, [layer(att(8, 2, 64, 0.125, (200000.0, 32), 50, dict(BANDS, factor=3.0)), moe(96, 8, 3)),
                            layer(att(3, 1, 96, 0.1, (1000.0, 96), 130), moe(64, 12, 2)), layer(att(2, 2, 128, 0.09, (1000.0, 128)), None)], side=40)
# the first layers looped twice from the embedding on, a second table whose part of a row is an odd number
CFG_FRONT = config(71, 96, [layer(att(6, 3, 32, 0.2, (5000.0, 16), 40), moe(32, 6, 1)), layer(att(2, 1, 32, 0.2, (5000.0, 32), 40, BANDS), None),
                            layer(att(2, 1, 32, 0.2, (5000.0, 16), 40), moe(56, 4, 2))], loop=(0, 2, 2), side=5, mult=0.45)

CONFIGS = {"all": CFG_ALL, "odd": CFG_ODD, "wide": CFG_WIDE, "front": CFG_FRONT}


def make_tensors(cfg, seed):
    """name -> float32 array, drawn so that every mechanism matters: norm weights and scales away from 1 (of both signs for the scales), biases away
    from 0, scores of order one and more, gates and router scores on both sides of a half, vectors in front of passes as large as the rows."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    n = lambda *shape, std=1.0: (rng.standard_normal(shape) * std).astype(np.float32)
    t = {"embed": n(V, W)}

    def norm(name):
        t[name], t[name + ".b"] = 1 + n(W, std=0.2), n(W, std=0.15)

    norm("final.norm")
    side = (cfg.get("token_side") or {}).get("dim")
    if side:
        t["side.embed"] = n(V, side * len(cfg["layers"]))
    if cfg.get("loop") is not None:
        t["loop.step"] = n(cfg["loop"]["times"], W, std=0.7)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q = p + "mix."
        norm(p + "norm1")
        t[q + "q"], t[q + "k"] = n(m["heads"] * m["dim"], W, std=1.5 * W ** -0.5), n(m["kv_heads"] * m["dim"], W, std=1.5 * W ** -0.5)
        t[q + "q.norm"], t[q + "k.norm"] = 1 + n(m["dim"], std=0.3), 1 + n(m["dim"], std=0.3)
        t[q + "g"], t[q + "o"] = n(m["heads"], W, std=2.0 * W ** -0.5), n(W, m["heads"] * m["dim"], std=(m["heads"] * m["dim"]) ** -0.5)
        t[p + "ls1"] = n(W, std=0.8)
        if l["mlp"] is not None:
            ff, r = l["mlp"]["expert"]["ff"], l["mlp"]["router"]
            norm(p + "norm2")
            for e in range(r["experts"]):
                t[f"{p}mlp.e{e}.up"], t[f"{p}mlp.e{e}.down"] = n(ff, W, std=1.6 * W ** -0.5), n(W, ff, std=ff ** -0.5)
            t[p + "mlp.router"], t[p + "ls2"] = n(r["experts"], W, std=2 * W ** -0.5), n(W, std=0.8)
        if side:
            t[p + "side.gate"], t[p + "side.proj"], t[p + "side.norm"] = n(side, W, std=1.2 * W ** -0.5), n(W, side, std=side ** -0.5), n(W, std=0.7)
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
