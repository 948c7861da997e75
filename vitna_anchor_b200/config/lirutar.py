"""Typed configuration of the Lirutar decoder, read from config.json.

config.json gives every size and every constant that differs between models of the design:

    architecture      "Lirutar"
    vocab, width
    norm.eps          eps of every norm of the model (the layer norms around the sublayers, the RMS norm inside the mixer)
    layers            a list; each entry has `type` (parallel), `mixer` (its sizes) and `mlp` (or null)
    loop              {start, stop, times}: layers start..stop-1 run `times` times in a row with the same weights, every pass with caches and
                      states of its own and with a product of [x | embedding output] in front (absent: every layer runs once, and there
                      is no such product)

A parallel mixer gives left {heads, kv_heads, dim, vdim, scale, rot {base, dims}, mask {size}}, right {heads, vdim, state, groups, conv,
norm_groups} and left_scale, right_scale.  kv_heads (heads), vdim (dim), rot (no rotation), mask (no window) may be left out, as may the two
scales (1), groups and norm_groups (1).  A feed-forward is {kind: dense, ff} or {kind: moe, expert {ff, limit}, router {experts, top, groups
{count, keep}, identity, scale}, shared {ff, limit}}; groups (one), identity (0), scale (1) and shared (none) may be left out.  There is no limit on
positions: nothing of the model is a table over them.  A key inside a layer that this reader does not know is refused by name.
"""
from __future__ import annotations

import warnings
from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .errors import ConfigError
from .lupanex import _known, _number, _size

ARCHITECTURE = "Lirutar"


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotation]
    window: int                         # 0: every earlier position is seen


@dataclass(frozen=True)
class StateSpaceSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class ParallelSpec:
    left: AttentionSpec
    right: StateSpaceSpec
    left_scale: float
    right_scale: float

    kind = "parallel"


@dataclass(frozen=True)
class DenseFFSpec:
    ff: int

    kind = "dense"


@dataclass(frozen=True)
class ExpertSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class ExpertsFFSpec:
    expert: ExpertSpec
    experts: int
    identity: int
    top: int
    count: int
    keep: int
    scale: float
    shared: Optional[ExpertSpec]

    kind = "moe"


@dataclass(frozen=True)
class LayerSpec:
    mixer: ParallelSpec
    mlp: Any                            # DenseFFSpec, ExpertsFFSpec or None


def _expert(entry: Any, where: str) -> ExpertSpec:
    _known(entry, where, ("ff", "limit"))
    limit = _number(entry, "limit", where + ".")
    if limit <= 0:
        raise ConfigError(f"config.json: {where}.limit is not positive")
    return ExpertSpec(_size(entry, "ff", where + "."), limit)


def _mlp(entry: Any, where: str):
    if entry is None:
        return None
    if not isinstance(entry, Mapping):
        raise ConfigError(f"config.json: {where} is not an object")
    kind = entry.get("kind")
    if kind == "dense":
        _known(entry, where, ("kind", "ff"))
        return DenseFFSpec(_size(entry, "ff", where + "."))
    if kind == "moe":
        _known(entry, where, ("kind", "expert", "router", "shared"))
        r, rw = entry.get("router"), where + ".router."
        _known(r, where + ".router", ("experts", "top", "groups", "identity", "scale"))
        experts, top = _size(r, "experts", rw), _size(r, "top", rw)
        identity = _size(r, "identity", rw, 0) if r.get("identity") is not None else 0
        count = keep = 1
        if r.get("groups") is not None:
            _known(r["groups"], rw + "groups", ("count", "keep"))
            count, keep = _size(r["groups"], "count", rw + "groups."), _size(r["groups"], "keep", rw + "groups.")
        if (experts + identity) % count:
            raise ConfigError(f"config.json: {rw}groups.count does not divide the experts and identities")
        if keep > count:
            raise ConfigError(f"config.json: {rw}groups.keep is larger than the number of groups")
        if top > (experts + identity) // count * keep or top > 32:
            raise ConfigError(f"config.json: {rw}top is larger than the number of experts that can be chosen (or than 32)")
        scale = _number(r, "scale", rw) if r.get("scale") is not None else 1.0
        shared = _expert(entry["shared"], where + ".shared") if entry.get("shared") is not None else None
        return ExpertsFFSpec(_expert(entry.get("expert"), where + ".expert"), experts, identity, top, count, keep, scale, shared)
    raise ConfigError(f"config.json: {where}.kind is {kind!r}; the kinds are dense and moe")


def _attention(m: Any, where: str) -> AttentionSpec:
    _known(m, where[:-1], ("heads", "kv_heads", "dim", "vdim", "scale", "rot", "mask"))
    heads, dim = _size(m, "heads", where), _size(m, "dim", where)
    kv = _size(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads do not divide into kv_heads groups")
    rot = None
    if m.get("rot") is not None:
        _known(m["rot"], where + "rot", ("base", "dims"))
        rot = Rotation(_number(m["rot"], "base", where + "rot."), _size(m["rot"], "dims", where + "rot.", 0))
        if rot.base <= 0 or rot.dims % 2 or rot.dims > dim:
            raise ConfigError(f"config.json: {where}rot needs a positive base and an even number of dims, at most dim")
    window = 0
    if m.get("mask") is not None:
        _known(m["mask"], where + "mask", ("size",))
        window = _size(m["mask"], "size", where + "mask.")
    scale = _number(m, "scale", where)
    if scale <= 0:
        raise ConfigError(f"config.json: {where}scale is not positive")
    return AttentionSpec(heads, kv, dim, _size(m, "vdim", where) if m.get("vdim") is not None else dim, scale, rot, window)


def _state_space(m: Any, where: str) -> StateSpaceSpec:
    _known(m, where[:-1], ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
    one = lambda k: _size(m, k, where) if m.get(k) is not None else 1
    spec = StateSpaceSpec(_size(m, "heads", where), _size(m, "vdim", where), _size(m, "state", where), one("groups"), _size(m, "conv", where), one("norm_groups"))
    if spec.heads % spec.groups:
        raise ConfigError(f"config.json: {where}heads do not divide into groups")
    if spec.heads * spec.vdim % spec.norm_groups:
        raise ConfigError(f"config.json: {where}norm_groups does not divide heads * vdim")
    return spec


def _layer(i: int, entry: Mapping[str, Any]) -> LayerSpec:
    where = f"layers[{i}]."
    _known(entry, f"layers[{i}]", ("type", "mixer", "mlp"))
    kind, m = entry.get("type"), entry.get("mixer")
    if kind != "parallel":
        raise ConfigError(f"config.json: {where}type is {kind!r}; the mixer is parallel")
    _known(m, where + "mixer", ("left", "right", "left_scale", "right_scale"))
    one = lambda k: _number(m, k, where + "mixer.") if m.get(k) is not None else 1.0
    return LayerSpec(ParallelSpec(_attention(m.get("left"), where + "mixer.left."), _state_space(m.get("right"), where + "mixer.right."),
                                  one("left_scale"), one("right_scale")), _mlp(entry.get("mlp"), f"layers[{i}].mlp"))


@dataclass(frozen=True)
class LirutarConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[Tuple[int, int, int]]            # (start, stop, times)

    architecture = ARCHITECTURE

    @classmethod
    def from_dict(cls, cfg: Mapping[str, Any]) -> "LirutarConfig":
        top = ("architecture", "architectures", "vocab", "width", "norm", "layers", "loop")
        other = sorted(set(cfg) - set(top))
        if other:       # notes beside the model (a name, a seed) are no part of it; a key inside a layer is, and is refused
            warnings.warn(f"config.json: keys that are no part of the model are ignored: {', '.join(other)}", stacklevel=2)
        _known(cfg.get("norm"), "norm", ("eps",))
        eps = _number(cfg["norm"], "eps", "norm.")
        if eps < 0:
            raise ConfigError("config.json: norm.eps is negative")
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
        return cls(vocab=_size(cfg, "vocab", ""), width=_size(cfg, "width", ""), eps=eps, layers=layers, loop=loop)

    def runs(self) -> List[Tuple[int, bool]]:
        """(layer, whether a pass over the looped layers begins with it) in the order they run, a looped layer as often as it runs."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        start, stop, times = self.loop
        one_pass = [(i, i == start) for i in range(start, stop)]
        return [(i, False) for i in range(start)] + one_pass * times + [(i, False) for i in range(stop, n)]

    def to_dict(self) -> dict:
        """The config.json that reads back as this configuration."""
        def mixer(m):
            l, r = m.left, m.right
            left = dict(heads=l.heads, kv_heads=l.kv_heads, dim=l.dim, vdim=l.vdim, scale=l.scale)
            if l.rot is not None:
                left["rot"] = dict(base=l.rot.base, dims=l.rot.dims)
            if l.window:
                left["mask"] = dict(size=l.window)
            return dict(left=left, right=dict(heads=r.heads, vdim=r.vdim, state=r.state, groups=r.groups, conv=r.conv, norm_groups=r.norm_groups),
                        left_scale=m.left_scale, right_scale=m.right_scale)

        def mlp(f):
            if f is None:
                return None
            if isinstance(f, DenseFFSpec):
                return dict(kind="dense", ff=f.ff)
            d = dict(kind="moe", expert=dict(ff=f.expert.ff, limit=f.expert.limit),
                     router=dict(experts=f.experts, top=f.top, groups=dict(count=f.count, keep=f.keep), identity=f.identity, scale=f.scale))
            if f.shared is not None:
                d["shared"] = dict(ff=f.shared.ff, limit=f.shared.limit)
            return d

        d = dict(architecture=ARCHITECTURE, vocab=self.vocab, width=self.width, norm=dict(eps=self.eps),
                 layers=[dict(type=l.mixer.kind, mixer=mixer(l.mixer), mlp=mlp(l.mlp)) for l in self.layers])
        if self.loop is not None:
            d["loop"] = dict(start=self.loop[0], stop=self.loop[1], times=self.loop[2])
        return d
