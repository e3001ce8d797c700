"""Typed configuration of the Fotulix decoder, read from config.json's own keys.

config.json names the width, the vocabulary, the norms' eps, the embedding's scale and its table of token pairs
(`embedding.scale`, `embedding.bigram`), the factor on every sublayer's normed output (`residual_mult`), the size of the
input by token in every layer (`token_side.dim`) and a list of layers; every layer names its mixer (`type`: `attention`,
`attention_2` or `latent_attention`), the mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`: `dense`, or null
for none).  Every size and constant is a field here.  What config.json leaves out does not exist in the model (no `mask`:
every earlier key is seen; no `kv_heads`: a key head a query head; no `q_temp`, no `rot`, no `scaling`: none; no `embedding`:
scale 1 and no pairs; no `residual_mult`: 1; no `token_side`: no such input).  An unknown mixer type or feed-forward kind is
an error, a key the engine does not know is named in a warning.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from .dirurax_config import _only
from .model_config import ConfigError, _eos_ids, _need
from .pikalix_config import _table


@dataclass(frozen=True)
class BandScaling:
    """Rotary frequencies scaled by the band of their wavelength: kept below original/high, divided by `factor` above
    original/low, blended between."""
    factor: float
    low: float
    high: float
    original: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "BandScaling":
        _only(d, ("factor", "low", "high", "original"), "a rotation's scaling")
        c = cls(*(_need(d, k, float) for k in ("factor", "low", "high", "original")))
        if not (c.factor > 0 and 0 < c.low < c.high and c.original > 0):
            raise ConfigError("config.json: a rotation's scaling needs factor > 0, 0 < low < high, original > 0")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}

    def rope_scaling(self) -> Dict[str, Any]:
        return {"rope_type": "llama3", "factor": self.factor, "low_freq_factor": self.low, "high_freq_factor": self.high,
                "original_max_position_embeddings": self.original}


@dataclass(frozen=True)
class RampScaling:
    """YaRN: frequencies divided by `factor` along a ramp over the pairs that turn between `slow` and `fast` times over
    `original` positions, cos and sin with a factor of their own."""
    factor: float
    original: float
    fast: float
    slow: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RampScaling":
        _only(d, ("factor", "original", "fast", "slow"), "a rotation's scaling")
        c = cls(*(_need(d, k, float) for k in ("factor", "original", "fast", "slow")))
        if not min(c.factor, c.original, c.fast, c.slow) > 0:
            raise ConfigError("config.json: a rotation's scaling needs positive numbers")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}

    def rope_scaling(self) -> Dict[str, Any]:
        return {"rope_type": "yarn", "factor": self.factor, "original_max_position_embeddings": self.original,
                "beta_fast": self.fast, "beta_slow": self.slow}


@dataclass(frozen=True)
class RotationConfig:
    """The first `dims` channels of a head turn in pairs (2i, 2i+1) by p * base^(-2i/dims), scaled where `scaling` is given."""
    base: float
    dims: int
    scaling: Optional[Union[BandScaling, RampScaling]] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], scaling) -> "RotationConfig":
        _only(d, ("base", "dims", "scaling"), "a rotation")
        s = _table(d, "scaling", "a rotation")
        c = cls(_need(d, "base", float), _need(d, "dims"), scaling.from_dict(s) if s is not None else None)
        if not c.base > 0 or c.dims < 0 or c.dims % 2 or (c.base == 1.0 and s is not None):
            raise ConfigError("config.json: a rotation needs a positive base and an even count of channels")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d


def _grouped_sizes(d: Mapping[str, Any]):
    heads, dim = _need(d, "heads"), _need(d, "dim")
    sizes = (heads, int(d["kv_heads"]) if d.get("kv_heads") is not None else heads, dim,
             int(d["vdim"]) if d.get("vdim") is not None else dim, _need(d, "scale", float))
    if min(sizes[:4]) <= 0 or heads % sizes[1]:
        raise ConfigError("config.json: an attention mixer needs positive sizes and heads a multiple of kv_heads")
    return sizes


@dataclass(frozen=True)
class BucketAttentionConfig:
    """`attention`: grouped-query attention with biased projections and without rotation; a learned bias by the distance's
    bucket (the rows are the tensor's, the last serves distances from `bias_max` on), queries multiplied by
    1 + coef ln(floor((p + 1) / every) + 1) where `q_temp` is given, a gate per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    temp_coef: Optional[float] = None
    temp_every: Optional[float] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "BucketAttentionConfig":
        where = "an attention mixer"
        _only(d, ("heads", "kv_heads", "dim", "vdim", "scale", "bias_max", "q_temp"), where)
        temp = _table(d, "q_temp", where)
        coef = every = None
        if temp is not None:
            _only(temp, ("coef", "every"), "a query temperature")
            coef, every = _need(temp, "coef", float), _need(temp, "every", float)
            if not every > 0:
                raise ConfigError("config.json: q_temp.every must be positive")
        c = cls(*_grouped_sizes(d), _need(d, "bias_max", float), coef, every)
        if not c.bias_max > 0:
            raise ConfigError("config.json: bias_max must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale, "bias_max": self.bias_max}
        if self.temp_every is not None:
            d["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return d


@dataclass(frozen=True)
class RotaryAttentionConfig:
    """`attention_2`: grouped-query attention with rotated queries and keys, a learned sink and a gate per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationConfig] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RotaryAttentionConfig":
        where = "an attention_2 mixer"
        _only(d, ("heads", "kv_heads", "dim", "vdim", "scale", "rot"), where)
        rot = _table(d, "rot", where)
        c = cls(*_grouped_sizes(d), RotationConfig.from_dict(rot, BandScaling) if rot is not None else None)
        if c.rot is not None and c.rot.dims > c.dim:
            raise ConfigError("config.json: rot.dims is at most the head's size")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class LatentConfig:
    """`latent_attention`: keys and values made from one cached vector of `kv_rank` channels per token plus `rot_dim` rotated
    key channels all heads share, a sliding window, a gate per head.  `kv_from`: the layer whose cached rows this one reads
    instead of making its own."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[RotationConfig] = None
    mask_size: Optional[int] = None
    kv_from: Optional[int] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "LatentConfig":
        where = "a latent attention mixer"
        _only(d, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot", "mask", "kv_from"), where)
        rot, mask = _table(d, "rot", where), _table(d, "mask", where)
        if mask is not None:
            _only(mask, ("size",), "an attention mask")
        c = cls(_need(d, "heads"), _need(d, "dim"), _need(d, "rot_dim"), _need(d, "vdim"), _need(d, "kv_rank"),
                _need(d, "scale", float), RotationConfig.from_dict(rot, RampScaling) if rot is not None else None,
                _need(mask, "size") if mask is not None else None, int(d["kv_from"]) if d.get("kv_from") is not None else None)
        if min(c.heads, c.dim, c.vdim, c.kv_rank) <= 0 or c.rot_dim < 0 or c.rot_dim % 2:
            raise ConfigError("config.json: a latent attention mixer needs positive sizes and an even rot_dim")
        if c.rot_dim and (c.rot is None or c.rot.dims != c.rot_dim):
            raise ConfigError("config.json: a latent attention mixer rotates its whole rotated part: rot.dims = rot_dim")
        if c.mask_size is not None and c.mask_size <= 0:
            raise ConfigError("config.json: mask.size must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim,
                             "kv_rank": self.kv_rank, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.mask_size is not None:
            d["mask"] = {"size": self.mask_size}
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "DenseConfig":
        _only(d, ("kind", "ff"), "a dense feed-forward")
        c = cls(_need(d, "ff"))
        if c.ff <= 0:
            raise ConfigError("config.json: a feed-forward needs a positive ff")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class BigramConfig:
    """Row (previous id * mul_prev + id * mul_cur) mod buckets of a table is added to a token's embedding."""
    buckets: int
    mul_prev: int
    mul_cur: int

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "BigramConfig":
        _only(d, ("buckets", "mul_prev", "mul_cur"), "a bigram embedding")
        c = cls(_need(d, "buckets"), _need(d, "mul_prev"), _need(d, "mul_cur"))
        if c.buckets <= 0 or min(c.mul_prev, c.mul_cur) < 0:
            raise ConfigError("config.json: a bigram embedding needs positive buckets and factors that are not negative")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}


MixerConfig = Union[BucketAttentionConfig, RotaryAttentionConfig, LatentConfig]
_MIXERS = {"attention": BucketAttentionConfig, "attention_2": RotaryAttentionConfig, "latent_attention": LatentConfig}
_MLPS = {"dense": DenseConfig}


@dataclass(frozen=True)
class FotulixLayer:
    type: str
    mixer: MixerConfig
    mlp: Optional[DenseConfig]

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], index: int) -> "FotulixLayer":
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
class FotulixConfig:
    width: int
    vocab: int
    norm_eps: float
    layers: Tuple[FotulixLayer, ...]
    embedding_scale: float = 1.0
    bigram: Optional[BigramConfig] = None
    residual_mult: float = 1.0
    side_dim: Optional[int] = None
    eos_token_ids: Tuple[int, ...] = ()
    architecture: str = "Fotulix"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], generation: Optional[Mapping[str, Any]] = None) -> "FotulixConfig":
        norm = d.get("norm")
        if not isinstance(norm, Mapping):
            raise ConfigError("config.json: required key 'norm' is missing")
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        emb, side = _table(d, "embedding", "the model"), _table(d, "token_side", "the model")
        bigram = None
        if emb is not None:
            _only(emb, ("scale", "bigram"), "the embedding")
            b = _table(emb, "bigram", "the embedding")
            bigram = BigramConfig.from_dict(b) if b is not None else None
        if side is not None:
            _only(side, ("dim",), "the input by token")
        vocab = _need(d, "vocab")
        cfg = cls(width=_need(d, "width"), vocab=vocab, norm_eps=_need(norm, "eps", float),
                  layers=tuple(FotulixLayer.from_dict(l, i) for i, l in enumerate(layers)),
                  embedding_scale=float(emb["scale"]) if emb is not None and emb.get("scale") is not None else 1.0,
                  bigram=bigram,
                  residual_mult=float(d["residual_mult"]) if d.get("residual_mult") is not None else 1.0,
                  side_dim=_need(side, "dim") if side is not None else None,
                  eos_token_ids=_eos_ids(d, generation, vocab),
                  architecture=str(d.get("architecture") or "Fotulix"))
        if cfg.width <= 0 or cfg.vocab <= 0 or not cfg.norm_eps > 0:
            raise ConfigError("config.json: width, vocab and norm.eps must be positive")
        if cfg.side_dim is not None and cfg.side_dim <= 0:
            raise ConfigError("config.json: token_side.dim must be positive")
        for i, layer in enumerate(cfg.layers):
            cfg._check_source(i, layer.mixer)
        return cfg

    def _check_source(self, i: int, m: MixerConfig) -> None:
        """A layer that reads another's cached rows: an earlier latent layer with rows of its own, of the same sizes and
        rotation."""
        if not isinstance(m, LatentConfig) or m.kv_from is None:
            return
        if not 0 <= m.kv_from < i:
            raise ConfigError(f"config.json: layer {i} reads the rows of layer {m.kv_from}, which does not run before it")
        src = self.layers[m.kv_from].mixer
        if not isinstance(src, LatentConfig) or src.kv_from is not None:
            raise ConfigError(f"config.json: layer {i} reads the rows of layer {m.kv_from}, which caches none of its own")
        if (src.kv_rank, src.rot_dim, src.rot) != (m.kv_rank, m.rot_dim, m.rot):
            raise ConfigError(f"config.json: layers {m.kv_from} and {i} share rows but differ in kv_rank, rot_dim or rot")

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab,
                             "norm": {"eps": self.norm_eps}, "layers": [l.to_dict() for l in self.layers]}
        emb: Dict[str, Any] = {}
        if self.embedding_scale != 1.0:
            emb["scale"] = self.embedding_scale
        if self.bigram is not None:
            emb["bigram"] = self.bigram.to_dict()
        if emb:
            d["embedding"] = emb
        if self.residual_mult != 1.0:
            d["residual_mult"] = self.residual_mult
        if self.side_dim is not None:
            d["token_side"] = {"dim": self.side_dim}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
