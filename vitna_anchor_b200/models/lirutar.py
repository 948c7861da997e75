"""The Lirutar decoder: manifest of its tensors and how its layers are built from the engine's parts.

A small decoder-only language model.  Token rows are normed before the first layer.  Every layer is pre-norm (layer norms with weight and bias):
its mixer is two mixers side by side on the same input, a grouped-query attention (biases, a partial rotation, values of their own size,
a window) and a state-space mixer (a matrix state per head behind a short convolution), each with a factor on its output; its feed-forward a
dense one with relu squared or routed experts (scores over experts and identities, a correction of the choice, groups, a shared expert),
or absent.  A range of layers may run several times in a row with the same weights, every pass with caches and states of its own and with a
product of [x | embedding output] in front.

Tensor names: embed, embed.norm(.b), loop.in, final.norm(.b), head; layer i has l<i>.norm1(.b), l<i>.norm2(.b), l<i>.mix.{left,right}.* and l<i>.mlp.*.
Matrices are [out, in].
"""
from __future__ import annotations

from typing import Dict, List

import numpy as np
import torch

from ..config.lirutar import DenseFFSpec, ExpertsFFSpec, LirutarConfig
from ..parts.embedding import LMHead, NormedEmbedding
from ..parts.feed_forward import ScoredRouter
from ..parts.loop import PassInput
from ..parts.registry import make_part
from ..weights.loader import WeightSpec
from .decoder import DecoderModel, LayerRun

UNBOUNDED_POSITIONS = 1 << 24       # nothing of the model is a table over positions; float32 holds these exactly
EXPERT_ALPHA = 1.702                # the sigmoid's factor in an expert's gate


def lirutar_manifest(cfg: LirutarConfig) -> List[WeightSpec]:
    W = cfg.width
    norm = lambda name: [WeightSpec(name, (W,)), WeightSpec(name + ".b", (W,))]
    gated = lambda q, ff: [WeightSpec(q + "gate", (ff, W)), WeightSpec(q + "up", (ff, W)), WeightSpec(q + "down", (W, ff))]
    m = [WeightSpec("embed", (cfg.vocab, W))] + norm("embed.norm")
    if cfg.loop is not None:
        m.append(WeightSpec("loop.in", (W, 2 * W)))
    for i, layer in enumerate(cfg.layers):
        p, l, r = f"l{i}.", layer.mixer.left, layer.mixer.right
        m += norm(p + "norm1")
        for name, rows in (("q", l.heads * l.dim), ("k", l.kv_heads * l.dim), ("v", l.kv_heads * l.vdim)):
            m += [WeightSpec(f"{p}mix.left.{name}", (rows, W)), WeightSpec(f"{p}mix.left.{name}.b", (rows,))]
        m.append(WeightSpec(p + "mix.left.o", (W, l.heads * l.vdim)))
        inner, channels = r.heads * r.vdim, r.heads * r.vdim + 2 * r.groups * r.state
        q = p + "mix.right."
        m += [WeightSpec(q + "in", (inner + channels + r.heads, W)), WeightSpec(q + "conv", (channels, r.conv)), WeightSpec(q + "conv.b", (channels,)),
              WeightSpec(q + "dt_bias", (r.heads,)), WeightSpec(q + "A_log", (r.heads,)), WeightSpec(q + "D", (r.heads,)),
              WeightSpec(q + "norm", (inner,)), WeightSpec(q + "o", (W, inner))]
        ff = layer.mlp
        if ff is None:
            continue
        m += norm(p + "norm2")
        if isinstance(ff, DenseFFSpec):
            m += [WeightSpec(p + "mlp.up", (ff.ff, W)), WeightSpec(p + "mlp.down", (W, ff.ff))]
        else:
            for e in range(ff.experts):
                m += gated(f"{p}mlp.e{e}.", ff.expert.ff)
            m += [WeightSpec(p + "mlp.router", (ff.experts + ff.identity, W)), WeightSpec(p + "mlp.correction", (ff.experts + ff.identity,))]
            if ff.shared is not None:
                m += gated(p + "mlp.shared.", ff.shared.ff)
    return m + norm("final.norm") + [WeightSpec("head", (cfg.vocab, W))]


def is_norm_weight(name: str) -> bool:
    """Tensors that random initialisation makes 1 + noise instead of noise around 0."""
    return name.rsplit(".", 1)[-1] in ("norm1", "norm2", "norm")


def _frequencies(base: float, dims: int) -> torch.Tensor:
    """f_i = base^(-2i/dims) for i < dims / 2, worked out in float64 and rounded once."""
    return torch.from_numpy(np.power(float(base), -2.0 * np.arange(dims // 2, dtype=np.float64) / float(dims)).astype(np.float32))


def build_lirutar(cfg: LirutarConfig, weights: Dict[str, torch.Tensor], dtype: torch.dtype, device) -> DecoderModel:
    """Matrices go to the device in the compute dtype; norms, biases, convolution weights, the heads' numbers, routers and corrections are
    float32 in both paths."""
    dev = torch.device(device)
    W = cfg.width

    def mat(*names: str) -> torch.Tensor:
        parts = [weights[n].to(device=dev, dtype=dtype) for n in names]
        return parts[0].contiguous() if len(parts) == 1 else torch.cat(parts, dim=0).contiguous()

    def vec(*names: str) -> torch.Tensor:
        parts = [weights[n].to(device=dev, dtype=torch.float32) for n in names]
        return parts[0].contiguous() if len(parts) == 1 else torch.cat(parts, dim=0).contiguous()

    def norm(name: str):
        return make_part("norm", "layernorm", width=W, eps=cfg.eps, weight=vec(name), bias=vec(name + ".b"))

    blocks = []
    for i, layer in enumerate(cfg.layers):
        p, l, r = f"l{i}.", layer.mixer.left, layer.mixer.right
        qkv = [f"{p}mix.left.{n}" for n in ("q", "k", "v")]
        dims = l.rot.dims if l.rot is not None else 0
        left = make_part("mixer", "rotary_attention", hidden=W, num_heads=l.heads, num_kv_heads=l.kv_heads, dim=l.dim, vdim=l.vdim, scale=l.scale,
                         w_in=mat(*qkv), w_out=mat(p + "mix.left.o"), b_in=vec(*[n + ".b" for n in qkv]),
                         freq=_frequencies(l.rot.base, dims).to(dev) if dims else None, rot_dims=dims, window=l.window)
        q = p + "mix.right."
        right = make_part("mixer", "ssd", hidden=W, num_heads=r.heads, groups=r.groups, state=r.state, vdim=r.vdim, taps=r.conv, w_in=mat(q + "in"),
                          conv=vec(q + "conv"), conv_b=vec(q + "conv.b"), dt_bias=vec(q + "dt_bias"), a_log=vec(q + "A_log"), D=vec(q + "D"),
                          norm_weight=vec(q + "norm"), norm_parts=r.norm_groups, w_out=mat(q + "o"), eps=cfg.eps)
        mixer = make_part("mixer", "parallel", left=left, right=right, left_scale=layer.mixer.left_scale, right_scale=layer.mixer.right_scale)
        ffn = ffn_norm = None
        ff = layer.mlp
        if isinstance(ff, DenseFFSpec):
            ffn = make_part("feed_forward", "dense", hidden=W, intermediate=ff.ff, w_up=mat(p + "mlp.up"), w_down=mat(p + "mlp.down"), activation="relu2")
        elif isinstance(ff, ExpertsFFSpec):
            shared = None
            if ff.shared is not None:
                s = p + "mlp.shared."
                shared = make_part("feed_forward", "clamped_glu", hidden=W, intermediate=ff.shared.ff, w_gate_up=mat(s + "gate", s + "up"),
                                   w_down=mat(s + "down"), limit=ff.shared.limit, alpha=EXPERT_ALPHA)
            ffn = make_part("feed_forward", "routed_experts", hidden=W, intermediate=ff.expert.ff, experts=ff.experts, top=ff.top, w_router=vec(p + "mlp.router"),
                            b_router=None, w_gate_up=torch.stack([mat(f"{p}mlp.e{e}.gate", f"{p}mlp.e{e}.up") for e in range(ff.experts)]).contiguous(),
                            w_down=torch.stack([mat(f"{p}mlp.e{e}.down") for e in range(ff.experts)]).contiguous(), shared=shared, activation="clamped",
                            limit=ff.expert.limit, alpha=EXPERT_ALPHA,
                            scored=ScoredRouter(vec(p + "mlp.correction"), ff.count, ff.keep, ff.identity, ff.scale))
        if ffn is not None:
            ffn_norm = norm(p + "norm2")
        blocks.append(make_part("block", "pre_norm", mixer_norm=norm(p + "norm1"), mixer=mixer, ffn_norm=ffn_norm, ffn=ffn))
    # every run of a layer, a looped one each time, has pages and a state of its own; the states come behind the pages' cache layers
    enter = PassInput(W, mat("loop.in")) if cfg.loop is not None else None
    runs = cfg.runs()
    schedule = [LayerRun(block=b, cache=n, state=len(runs) + n, before=enter if begins else None) for n, (b, begins) in enumerate(runs)]
    embedding = NormedEmbedding(cfg.vocab, W, mat("embed"), norm("embed.norm"))
    return DecoderModel(embedding=embedding, blocks=blocks, schedule=schedule, final_norm=norm("final.norm"), lm_head=LMHead(cfg.vocab, W, mat("head")),
                        position=None, dtype=dtype, vocab_size=cfg.vocab, max_positions=UNBOUNDED_POSITIONS, config=cfg)
