"""Typed configuration of the Zolapel decoder, read from config.json.

config.json gives every size and every constant that differs between models of the design:

    architecture      "Zolapel"
    vocab, width
    norm.eps          eps of every norm of the model (layer norms around the sublayers, RMS norms of queries, keys and per-layer inputs)
    residual_mult     the factor on everything that is added to the residual stream (absent: 1)
    token_side.dim    the part of a token's row of the second table that each layer reads (absent: no such inputs)
    layers            a list; each entry has `type` (attention), `mixer` (its sizes) and `mlp` (or null)
    loop              {start, stop, times}: layers start..stop-1 run `times` times in a row with the same weights, every pass with a cache of
                      its own, with a vector of its own and, but for the first, the embedding output added in front (absent: every layer
                      runs once, and there are no such vectors)

An attention gives heads, kv_heads, dim, vdim, scale, rot {base, dims, scaling {factor, low, high, original}} and mask {size}; kv_heads (heads),
vdim (dim, the only value it can have: the values are the projected keys), rot (no rotation), scaling (none) and mask (no window) may be left out.
A feed-forward is {kind: moe, expert {ff}, router {experts, top}}.  There is no limit on positions: nothing of the model is a table over them.
A key inside a layer that this reader does not know is refused by name.
"""
from __future__ import annotations

import warnings
from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .errors import ConfigError
from .lupanex import _known, _number, _size

ARCHITECTURE = "Zolapel"


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int
    scaling: Optional[Tuple[float, float, float, float]] = None         # (factor, low, high, original)


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot: Optional[Rotation]
    window: int                         # 0: every earlier position is seen

    kind = "attention"


@dataclass(frozen=True)
class ExpertsFFSpec:
    ff: int
    experts: int
    top: int

    kind = "moe"


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec
    mlp: Optional[ExpertsFFSpec]


def _rotation(entry: Any, where: str, dim: int) -> Rotation:
    _known(entry, where, ("base", "dims", "scaling"))
    base, dims = _number(entry, "base", where + "."), _size(entry, "dims", where + ".", 0)
    if base <= 0 or dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where} needs a positive base and an even number of dims, at most dim")
    scaling = None
    if entry.get("scaling") is not None:
        at = where + ".scaling"
        _known(entry["scaling"], at, ("factor", "low", "high", "original"))
        scaling = tuple(_number(entry["scaling"], k, at + ".") for k in ("factor", "low", "high", "original"))
        if min(scaling) <= 0 or scaling[1] > scaling[2]:
            raise ConfigError(f"config.json: {at} needs positive numbers, low at most high")
    return Rotation(base, dims, scaling)


def _attention(m: Any, where: str) -> AttentionSpec:
    _known(m, where[:-1], ("heads", "kv_heads", "dim", "vdim", "scale", "rot", "mask"))
    heads, dim = _size(m, "heads", where), _size(m, "dim", where)
    kv = _size(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads do not divide into kv_heads groups")
    if m.get("vdim") is not None and _size(m, "vdim", where) != dim:
        raise ConfigError(f"config.json: {where}vdim is not dim; the values are the projected keys")
    window = 0
    if m.get("mask") is not None:
        _known(m["mask"], where + "mask", ("size",))
        window = _size(m["mask"], "size", where + "mask.")
    scale = _number(m, "scale", where)
    if scale <= 0:
        raise ConfigError(f"config.json: {where}scale is not positive")
    return AttentionSpec(heads, kv, dim, scale, _rotation(m["rot"], where + "rot", dim) if m.get("rot") is not None else None, window)


def _mlp(entry: Any, where: str) -> Optional[ExpertsFFSpec]:
    if entry is None:
        return None
    if not isinstance(entry, Mapping) or entry.get("kind") != "moe":
        raise ConfigError(f"config.json: {where} is not a feed-forward of the kind moe")
    _known(entry, where, ("kind", "expert", "router"))
    _known(entry.get("expert"), where + ".expert", ("ff",))
    _known(entry.get("router"), where + ".router", ("experts", "top"))
    spec = ExpertsFFSpec(_size(entry["expert"], "ff", where + ".expert."), _size(entry["router"], "experts", where + ".router."),
                         _size(entry["router"], "top", where + ".router."))
    if spec.top > min(spec.experts, 32):
        raise ConfigError(f"config.json: {where}.router.top is larger than the number of experts (or than 32)")
    return spec


def _layer(i: int, entry: Mapping[str, Any]) -> LayerSpec:
    where = f"layers[{i}]"
    _known(entry, where, ("type", "mixer", "mlp"))
    if entry.get("type") != "attention":
        raise ConfigError(f"config.json: {where}.type is {entry.get('type')!r}; the mixer is attention")
    return LayerSpec(_attention(entry.get("mixer"), where + ".mixer."), _mlp(entry.get("mlp"), where + ".mlp"))


@dataclass(frozen=True)
class ZolapelConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    side_dim: int                                   # 0: the layers read nothing from a second table
    layers: Tuple[LayerSpec, ...]
    loop: Optional[Tuple[int, int, int]]            # (start, stop, times)

    architecture = ARCHITECTURE

    @classmethod
    def from_dict(cls, cfg: Mapping[str, Any]) -> "ZolapelConfig":
        top = ("architecture", "architectures", "vocab", "width", "norm", "residual_mult", "token_side", "layers", "loop")
        other = sorted(set(cfg) - set(top))
        if other:       # notes beside the model (a name, a seed) are no part of it; a key inside a layer is, and is refused
            warnings.warn(f"config.json: keys that are no part of the model are ignored: {', '.join(other)}", stacklevel=2)
        _known(cfg.get("norm"), "norm", ("eps",))
        eps = _number(cfg["norm"], "eps", "norm.")
        if eps < 0:
            raise ConfigError("config.json: norm.eps is negative")
        side = 0
        if cfg.get("token_side") is not None:
            _known(cfg["token_side"], "token_side", ("dim",))
            side = _size(cfg["token_side"], "dim", "token_side.")
        entries = cfg.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: layers is not a list of layers")
        layers = tuple(_layer(i, e) for i, e in enumerate(entries))
        loop = None
        if cfg.get("loop") is not None:
            _known(cfg["loop"], "loop", ("start", "stop", "times"))
            loop = (_size(cfg["loop"], "start", "loop.", 0), _size(cfg["loop"], "stop", "loop.", 1), _size(cfg["loop"], "times", "loop."))
            if not loop[0] < loop[1] <= len(layers):
                raise ConfigError("config.json: loop.start .. loop.stop is not a range of the layers")
        mult = _number(cfg, "residual_mult", "") if cfg.get("residual_mult") is not None else 1.0
        return cls(vocab=_size(cfg, "vocab", ""), width=_size(cfg, "width", ""), eps=eps, residual_mult=mult, side_dim=side, layers=layers, loop=loop)

    def runs(self) -> List[Tuple[int, int]]:
        """(layer, the number of the pass over the looped layers that begins with this run, or -1) in the order they run, a looped layer as
        often as it runs."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, -1) for i in range(n)]
        start, stop, times = self.loop
        passes = [(i, t if i == start else -1) for t in range(times) for i in range(start, stop)]
        return [(i, -1) for i in range(start)] + passes + [(i, -1) for i in range(stop, n)]

    def to_dict(self) -> dict:
        """The config.json that reads back as this configuration."""
        def mixer(m):
            d = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.dim, scale=m.scale)
            if m.rot is not None:
                d["rot"] = dict(base=m.rot.base, dims=m.rot.dims)
                if m.rot.scaling is not None:
                    d["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), m.rot.scaling))
            if m.window:
                d["mask"] = dict(size=m.window)
            return d

        mlp = lambda f: None if f is None else dict(kind="moe", expert=dict(ff=f.ff), router=dict(experts=f.experts, top=f.top))
        d = dict(architecture=ARCHITECTURE, vocab=self.vocab, width=self.width, norm=dict(eps=self.eps), residual_mult=self.residual_mult,
                 layers=[dict(type=l.mixer.kind, mixer=mixer(l.mixer), mlp=mlp(l.mlp)) for l in self.layers])
        if self.side_dim:
            d["token_side"] = dict(dim=self.side_dim)
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d
