"""The Zolapel decoder: manifest of its tensors and how its layers are built from the engine's parts.

A small decoder-only language model.  Every layer is pre-norm (layer norms with weight and bias): a grouped-query attention whose values are the
projected keys (queries and keys normed per head, neighbouring pairs turned, a window, a gate a head), routed experts with relu squared whose inputs
the router's sigmoids multiply (or no feed-forward), each sublayer's result scaled value by value; at its end every layer reads a part of its own of
the token's row of a second table.  A range of layers may run several times in a row with the same weights, every pass with a cache of its own, with
a vector of its own and, but for the first, the embedding output added in front.  The embedding table is the output matrix.

Tensor names: embed, side.embed, loop.step, final.norm(.b); layer i has l<i>.norm1(.b), l<i>.norm2(.b), l<i>.mix.*, l<i>.mlp.*, l<i>.ls1, l<i>.ls2 and
l<i>.side.*.  Matrices are [out, in].
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..config.zolapel import ZolapelConfig
from ..parts.block import ScaledResidualFlush, TokenSide
from ..parts.embedding import Embedding, LMHead
from ..parts.feed_forward import ScoredRouter
from ..parts.loop import PassOffset
from ..parts.registry import make_part
from ..parts.rotary import banded_frequencies
from ..weights.loader import WeightSpec
from .decoder import DecoderModel, LayerRun

UNBOUNDED_POSITIONS = 1 << 24       # nothing of the model is a table over positions; float32 holds these exactly


def zolapel_manifest(cfg: ZolapelConfig) -> List[WeightSpec]:
    W = cfg.width
    norm = lambda name: [WeightSpec(name, (W,)), WeightSpec(name + ".b", (W,))]
    m = [WeightSpec("embed", (cfg.vocab, W))]
    if cfg.loop is not None:
        m.append(WeightSpec("loop.step", (cfg.loop[2], W)))
    if cfg.side_dim:
        m.append(WeightSpec("side.embed", (cfg.vocab, len(cfg.layers) * cfg.side_dim)))
    for i, layer in enumerate(cfg.layers):
        p, a, ff = f"l{i}.", layer.mixer, layer.mlp
        q = p + "mix."
        m += norm(p + "norm1")
        m += [WeightSpec(q + "q", (a.heads * a.dim, W)), WeightSpec(q + "k", (a.kv_heads * a.dim, W)), WeightSpec(q + "q.norm", (a.dim,)),
              WeightSpec(q + "k.norm", (a.dim,)), WeightSpec(q + "g", (a.heads, W)), WeightSpec(q + "o", (W, a.heads * a.dim)), WeightSpec(p + "ls1", (W,))]
        if ff is not None:
            m += norm(p + "norm2")
            for e in range(ff.experts):
                m += [WeightSpec(f"{p}mlp.e{e}.up", (ff.ff, W)), WeightSpec(f"{p}mlp.e{e}.down", (W, ff.ff))]
            m += [WeightSpec(p + "mlp.router", (ff.experts, W)), WeightSpec(p + "ls2", (W,))]
        if cfg.side_dim:
            m += [WeightSpec(p + "side.gate", (cfg.side_dim, W)), WeightSpec(p + "side.proj", (W, cfg.side_dim)), WeightSpec(p + "side.norm", (W,))]
    return m + norm("final.norm")


def is_norm_weight(name: str) -> bool:
    """Tensors that random initialisation makes 1 + noise instead of noise around 0: the norms' weights and the sublayers' scales."""
    return name.rsplit(".", 1)[-1] in ("norm1", "norm2", "norm", "ls1", "ls2")


def build_zolapel(cfg: ZolapelConfig, weights: Dict[str, torch.Tensor], dtype: torch.dtype, device) -> DecoderModel:
    """Matrices and tables go to the device in the compute dtype; norms, scales, the passes' vectors and routers are float32 in both paths.  The factor on
    everything that is added is folded into the sublayers' float32 scales."""
    dev = torch.device(device)
    W = cfg.width

    def mat(*names: str) -> torch.Tensor:
        parts = [weights[n].to(device=dev, dtype=dtype) for n in names]
        return parts[0].contiguous() if len(parts) == 1 else torch.cat(parts, dim=0).contiguous()

    def vec(name: str) -> torch.Tensor:
        return weights[name].to(device=dev, dtype=torch.float32).contiguous()

    def norm(name: str):
        return make_part("norm", "layernorm", width=W, eps=cfg.eps, weight=vec(name), bias=vec(name + ".b"))

    table = mat("embed")
    side_table = mat("side.embed") if cfg.side_dim else None
    blocks = []
    for i, layer in enumerate(cfg.layers):
        p, a, ff = f"l{i}.", layer.mixer, layer.mlp
        q = p + "mix."
        dims = a.rot.dims if a.rot is not None else 0
        freq = torch.from_numpy(banded_frequencies(a.rot.base, dims, a.rot.scaling)).to(dev) if dims else None
        mixer = make_part("mixer", "rotary_attention", hidden=W, num_heads=a.heads, num_kv_heads=a.kv_heads, dim=a.dim, vdim=a.dim, scale=a.scale,
                          w_in=mat(q + "q", q + "k", q + "g"), w_out=mat(q + "o"), freq=freq, rot_dims=dims, window=a.window, eps=cfg.eps,
                          q_norm=vec(q + "q.norm"), k_norm=vec(q + "k.norm"), neighbours=True, v_from_k=True, gate=True)
        half = {}
        if ff is not None:
            ups, downs = ([mat(f"{p}mlp.e{e}.{n}") for e in range(ff.experts)] for n in ("up", "down"))
            half = dict(ffn_norm=norm(p + "norm2"), ffn_scale=cfg.residual_mult * vec(p + "ls2"),
                        ffn=make_part("feed_forward", "routed_experts", hidden=W, intermediate=ff.ff, experts=ff.experts, top=ff.top,
                                      w_router=vec(p + "mlp.router"), b_router=None, w_gate_up=torch.stack(ups).contiguous(),
                                      w_down=torch.stack(downs).contiguous(), activation="relu2", gated=False, weigh_input=True,
                                      scored=ScoredRouter(sigmoid=True)))
        side = None
        if cfg.side_dim:
            side = TokenSide(W, mat(p + "side.gate"), mat(p + "side.proj"), side_table, i * cfg.side_dim, vec(p + "side.norm"), cfg.eps, cfg.residual_mult)
        blocks.append(make_part("block", "scaled_residual", mixer_norm=norm(p + "norm1"), mixer=mixer, mixer_scale=cfg.residual_mult * vec(p + "ls1"),
                                side=side, **half))
    # every run of a layer, a looped one each time, has pages of its own
    enter = {}
    if cfg.loop is not None:
        steps = vec("loop.step")
        enter = {t: PassOffset(W, steps[t], table if t > 0 else None, deferred=True) for t in range(cfg.loop[2])}
    schedule = [LayerRun(block=b, cache=n, before=enter.get(t)) for n, (b, t) in enumerate(cfg.runs())]
    return DecoderModel(embedding=Embedding(cfg.vocab, W, table), blocks=blocks, schedule=schedule, final_norm=norm("final.norm"),
                        lm_head=LMHead(cfg.vocab, W, table), position=None, dtype=dtype, vocab_size=cfg.vocab, max_positions=UNBOUNDED_POSITIONS, config=cfg,
                        collect=ScaledResidualFlush(cfg.eps))
