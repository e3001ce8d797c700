"""Typed configuration of the Dozotar decoder, read from config.json's own keys.

config.json names the width, the vocabulary, the norms' eps and a list of layers; every layer names its mixer (`type`:
`attention`, `retention` or `mamba2`), the mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`: `dense`,
`moe`, or null for none).  Every size and constant is a field here.  What config.json leaves out does not exist in the
model (no `mask`: every earlier key is seen; no `kv_heads`: a key head a query head; no `vdim`: values of the keys'
size; no `rot`: no rotation; no `groups` of a router: every expert can be chosen; no `shared`: no shared expert).  The
rows of the attention's bias table are the tensor's.  An unknown mixer type or feed-forward kind is an error, a key
the engine does not know is named in a warning.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from .dirurax_config import _only
from .model_config import ConfigError, _eos_ids, _need
from .pikalix_config import _table


def _int(d: Mapping[str, Any], key: str, default: int) -> int:
    return int(d[key]) if d.get(key) is not None else default


@dataclass(frozen=True)
class BucketAttentionConfig:
    """Grouped-query attention without rotation: short convolutions of `conv` taps on q, k and v, a learned bias by the
    distance's bucket that reaches its last row at `bias_max`, keys of the query's own chunk of `mask_size` positions."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    bias_max: float
    mask_size: Optional[int] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "BucketAttentionConfig":
        where = "an attention mixer"
        _only(d, ("heads", "kv_heads", "dim", "vdim", "conv", "scale", "bias_max", "mask"), where)
        mask = _table(d, "mask", where)
        if mask is not None:
            _only(mask, ("size",), "an attention mask")
        heads, dim = _need(d, "heads"), _need(d, "dim")
        c = cls(heads, _int(d, "kv_heads", heads), dim, _int(d, "vdim", dim), _need(d, "conv"), _need(d, "scale", float),
                _need(d, "bias_max", float), _need(mask, "size") if mask is not None else None)
        if min(c.heads, c.kv_heads, c.dim, c.vdim, c.conv) <= 0 or c.heads % c.kv_heads:
            raise ConfigError("config.json: an attention mixer needs positive sizes and heads a multiple of kv_heads")
        if not c.bias_max > 0 or (c.mask_size is not None and c.mask_size <= 0):
            raise ConfigError("config.json: bias_max and mask.size must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "conv": self.conv, "scale": self.scale, "bias_max": self.bias_max}
        if self.mask_size is not None:
            d["mask"] = {"size": self.mask_size}
        return d


@dataclass(frozen=True)
class RetentionConfig:
    """Linear attention with one fixed decay a head; q and k rotated on their first `rot_dims` channels."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot_dims: int = 0
    rot_base: float = 10000.0

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RetentionConfig":
        where = "a retention mixer"
        _only(d, ("heads", "dim", "vdim", "decay", "rot"), where)
        rot = _table(d, "rot", where)
        if rot is not None:
            _only(rot, ("base", "dims"), "a rotation")
        heads, dim = _need(d, "heads"), _need(d, "dim")
        decay = d.get("decay")
        if not isinstance(decay, (list, tuple)) or len(decay) != heads:
            raise ConfigError(f"config.json: a retention mixer lists a decay for each of its {heads} heads")
        c = cls(heads, dim, _int(d, "vdim", dim), tuple(float(x) for x in decay),
                _int(rot, "dims", dim) if rot is not None else 0, _need(rot, "base", float) if rot is not None else 10000.0)
        if min(c.heads, c.dim, c.vdim) <= 0 or not 0 <= c.rot_dims <= c.dim or c.rot_dims % 2 or not c.rot_base > 0:
            raise ConfigError("config.json: a retention mixer needs positive sizes and an even rot.dims of at most dim")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        if self.rot_dims:
            d["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
        return d


@dataclass(frozen=True)
class StateSpaceConfig:
    """Mamba-2: `heads` heads of `vdim` channels, a state of `state` rows a channel, input and output vectors shared by the
    heads of a group, a convolution of `conv` taps, the output normed in `norm_groups` parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "StateSpaceConfig":
        _only(d, ("heads", "vdim", "state", "groups", "conv", "norm_groups"), "a mamba2 mixer")
        c = cls(_need(d, "heads"), _need(d, "vdim"), _need(d, "state"), _int(d, "groups", 1), _need(d, "conv"),
                _int(d, "norm_groups", 1))
        if min(c.heads, c.vdim, c.state, c.groups, c.conv, c.norm_groups) <= 0 or c.heads % c.groups \
                or (c.heads * c.vdim) % c.norm_groups:
            raise ConfigError("config.json: a mamba2 mixer needs positive sizes, heads a multiple of groups and "
                              "heads * vdim a multiple of norm_groups")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "DenseConfig":
        _only(d, ("kind", "ff"), "a dense feed-forward")
        c = cls(_need(d, "ff"))
        if c.ff <= 0:
            raise ConfigError("config.json: a feed-forward's ff must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class GroupedExpertsConfig:
    """`experts` gated feed-forwards of `ff` channels, a token uses `top`, chosen among the `groups_keep` best of
    `groups_count` groups of neighbours (0: no groups); a shared expert of `shared_ff` channels (None: none)."""
    ff: int
    experts: int
    top: int
    groups_count: int = 0
    groups_keep: int = 0
    shared_ff: Optional[int] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "GroupedExpertsConfig":
        where = "a feed-forward of experts"
        _only(d, ("kind", "expert", "router", "shared"), where)
        expert, router, shared = _table(d, "expert", where), _table(d, "router", where), _table(d, "shared", where)
        if expert is None or router is None:
            raise ConfigError("config.json: a feed-forward of experts names its 'expert' and its 'router'")
        _only(expert, ("ff",), "an expert")
        _only(router, ("experts", "top", "groups"), "a router")
        groups = _table(router, "groups", "a router")
        if groups is not None:
            _only(groups, ("count", "keep"), "a router's groups")
        if shared is not None:
            _only(shared, ("ff",), "a shared expert")
        c = cls(_need(expert, "ff"), _need(router, "experts"), _need(router, "top"),
                _need(groups, "count") if groups is not None else 0, _need(groups, "keep") if groups is not None else 0,
                _need(shared, "ff") if shared is not None else None)
        if c.ff <= 0 or (c.shared_ff is not None and c.shared_ff <= 0) or not 1 <= c.top <= c.experts:
            raise ConfigError("config.json: experts need a positive ff and 1 <= top <= experts")
        if groups is not None and (c.groups_count <= 0 or c.experts % c.groups_count or not 1 <= c.groups_keep <= c.groups_count
                                   or c.groups_keep * (c.experts // c.groups_count) < c.top):
            raise ConfigError("config.json: groups.count divides the experts, and the groups kept hold at least `top` of them")
        return c

    def to_dict(self) -> Dict[str, Any]:
        router: Dict[str, Any] = {"experts": self.experts, "top": self.top}
        if self.groups_count:
            router["groups"] = {"count": self.groups_count, "keep": self.groups_keep}
        d: Dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": router}
        if self.shared_ff is not None:
            d["shared"] = {"ff": self.shared_ff}
        return d


MixerConfig = Union[BucketAttentionConfig, RetentionConfig, StateSpaceConfig]
MlpConfig = Union[DenseConfig, GroupedExpertsConfig]
_MIXERS = {"attention": BucketAttentionConfig, "retention": RetentionConfig, "mamba2": StateSpaceConfig}
_MLPS = {"dense": DenseConfig, "moe": GroupedExpertsConfig}


@dataclass(frozen=True)
class DozotarLayer:
    type: str
    mixer: MixerConfig
    mlp: Optional[MlpConfig]

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], index: int) -> "DozotarLayer":
        _only(d, ("type", "mixer", "mlp"), f"layer {index}")
        kind = d.get("type")
        if kind not in _MIXERS:
            raise ConfigError(f"config.json: layer {index} has mixer type {kind!r}; known: {sorted(_MIXERS)}")
        if not isinstance(d.get("mixer"), Mapping):
            raise ConfigError(f"config.json: layer {index} has no 'mixer'")
        mlp = _table(d, "mlp", f"layer {index}")
        if mlp is not None and mlp.get("kind") not in _MLPS:
            raise ConfigError(f"config.json: layer {index}: feed-forward kind {mlp.get('kind')!r} is not built; "
                              f"known: {sorted(_MLPS)}")
        return cls(kind, _MIXERS[kind].from_dict(d["mixer"]),
                   _MLPS[mlp["kind"]].from_dict(mlp) if mlp is not None else None)

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp else None}


@dataclass(frozen=True)
class DozotarConfig:
    width: int
    vocab: int
    norm_eps: float
    layers: Tuple[DozotarLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()
    architecture: str = "Dozotar"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], generation: Optional[Mapping[str, Any]] = None) -> "DozotarConfig":
        norm = d.get("norm")
        if not isinstance(norm, Mapping):
            raise ConfigError("config.json: required key 'norm' is missing")
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        vocab = _need(d, "vocab")
        cfg = cls(width=_need(d, "width"), vocab=vocab, norm_eps=_need(norm, "eps", float),
                  layers=tuple(DozotarLayer.from_dict(l, i) for i, l in enumerate(layers)),
                  eos_token_ids=_eos_ids(d, generation, vocab), architecture=str(d.get("architecture") or "Dozotar"))
        if cfg.width <= 0 or cfg.vocab <= 0 or not cfg.norm_eps > 0:
            raise ConfigError("config.json: width, vocab and norm.eps must be positive")
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab,
                             "norm": {"eps": self.norm_eps}, "layers": [l.to_dict() for l in self.layers]}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
