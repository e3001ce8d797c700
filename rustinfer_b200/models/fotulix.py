"""The Fotulix decoder as a registry entry: configuration -> model spec.

A token embedding times a scale plus a row for the pair of the previous token and this one; layers in the order config.json
lists them, each with an RMS norm (weights stored around zero) before and after each sublayer and the factor
`residual_mult` on what is added (the `sandwich` arrangement), and behind the feed-forward an input by token: a vector of
the token's own for this layer, gated by the stream.  Three kinds of mixer: `attention` (no rotation, a bias by the
distance's bucket, a query temperature, biased projections), `attention_2` (rotary pairs with Llama 3's frequency bands,
a sink a head) and `latent_attention` (keys and values from one cached low-rank vector a token, rotary pairs with YaRN's
ramp, a sliding window; a layer may read the rows another one cached); all with a gate a head.  The feed-forward is gated
by silu, the head has a matrix of its own.  Nothing here computes: the spec names registered parts and hands them the
numbers of config.json.

Tensor names: `embed`, `bigram`, `side.embed`, `head`, `final.norm`, and per layer i `l<i>.norm1`, `l<i>.norm1b`,
`l<i>.norm2`, `l<i>.norm2b`, `l<i>.mix.*` (a projection's bias and norm weight with `.b` and `.norm` added to its name),
`l<i>.mlp.gate|up|down`, `l<i>.side.gate|proj|norm`.
"""
from __future__ import annotations

from typing import Optional

from ..config.fotulix_config import BucketAttentionConfig, FotulixConfig, LatentConfig, RotaryAttentionConfig
from ..config.registry import ArchitectureFamily, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def _kept_window(cfg: FotulixConfig, owner: int) -> Optional[int]:
    """Rows the cache of latent layer `owner` must keep: the widest window among the layers that read it (None as soon as
    one of them sees every row)."""
    sizes = [l.mixer.mask_size for i, l in enumerate(cfg.layers)
             if i == owner or (isinstance(l.mixer, LatentConfig) and l.mixer.kv_from == owner)]
    return None if any(s is None for s in sizes) else max(sizes)


def _mixer_spec(cfg: FotulixConfig, i: int) -> PartSpec:
    m = cfg.layers[i].mixer
    if isinstance(m, BucketAttentionConfig):
        temp = None
        if m.temp_every is not None:
            temp = PartSpec("query_temperature", {"coef": m.temp_coef, "every": m.temp_every})
        return PartSpec("gated_attention", {
            "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
            "scale": m.scale, "bias": "buckets", "bias_far": m.bias_max, "proj_bias": True, "q_temperature": temp,
            "head_gate": True})
    if isinstance(m, RotaryAttentionConfig):
        rope = None
        if m.rot is not None and m.rot.dims:
            rope = PartSpec("rope", {"head_dim": m.dim, "rotary_dim": m.rot.dims, "theta": m.rot.base, "layout": "interleaved",
                                     "scaling": m.rot.scaling.rope_scaling() if m.rot.scaling else None})
        return PartSpec("gated_attention", {
            "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
            "scale": m.scale, "bias": "none", "position": rope, "sink": True, "head_gate": True})
    if isinstance(m, LatentConfig):
        scaling = m.rot.scaling.rope_scaling() if m.rot is not None and m.rot.scaling else None
        return PartSpec("latent_attention", {
            "hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim,
            "kv_rank": m.kv_rank, "scale": m.scale, "rot_base": m.rot.base if m.rot is not None else 10000.0,
            "rot_layout": "interleaved", "rot_scaling": scaling, "norm_eps": cfg.norm_eps, "gate": "head",
            "window": m.mask_size, "cache_window": _kept_window(cfg, i if m.kv_from is None else m.kv_from),
            "own_kv": m.kv_from is None})
    raise TypeError(f"no mixer for {type(m).__name__}")


def fotulix_model_spec(cfg: FotulixConfig) -> ModelSpec:
    layers, order = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."

        def norm(name: str, scale: float = 1.0, offset: float = 1.0) -> PartSpec:
            return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": name, "offset": offset,
                                        "scale": scale})
        extra = {"post_mixer_norm": norm("norm1b", cfg.residual_mult)}
        names = {"mixer": p + "mix.", "mixer_norm": p, "post_mixer_norm": p}
        ffn = side = None
        if layer.mlp is not None:
            ffn = PartSpec("swiglu", {"hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "output": "float32",
                                      "gate_name": "gate", "up_name": "up", "down_name": "down"})
            extra["post_ffn_norm"] = norm("norm2b", cfg.residual_mult)
            names.update({"ffn": p + "mlp.", "ffn_norm": p, "post_ffn_norm": p})
        if cfg.side_dim is not None:
            side = PartSpec("token_input", {
                "hidden_size": cfg.width, "vocab_size": cfg.vocab, "dim": cfg.side_dim,
                "table_columns": cfg.side_dim * len(cfg.layers), "column": i * cfg.side_dim, "table_name": "side.embed",
                "gate_name": p + "side.gate", "proj_name": p + "side.proj"})
            extra["post_side_norm"] = norm("side.norm", cfg.residual_mult, offset=0.0)
            names.update({"side": "", "post_side_norm": p})
        layers.append(LayerSpec(mixer=_mixer_spec(cfg, i), mixer_norm=norm("norm1"), ffn=ffn,
                                ffn_norm=norm("norm2") if ffn else None, side=side, names=names, arrangement="sandwich",
                                extra_norms=extra))
        order.append(RunEntry(i, layer.mixer.kv_from if isinstance(layer.mixer, LatentConfig) else None))
    stem = {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "scale": cfg.embedding_scale, "weight_name": "embed"}
    if cfg.bigram is not None:
        embed = PartSpec("bigram_embedding", {**stem, "buckets": cfg.bigram.buckets, "mul_prev": cfg.bigram.mul_prev,
                                              "mul_cur": cfg.bigram.mul_cur, "bigram_name": "bigram"})
    else:
        embed = PartSpec("scaled_embedding", stem)
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, layers=tuple(layers), run_order=tuple(order),
        final_norm=PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": "", "offset": 1.0}),
        embed_name="", final_norm_name="final.norm", head_name="head", tie_head=False, eos_token_ids=cfg.eos_token_ids,
        embed=embed, head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight_name": ""}))


FOTULIX = ArchitectureFamily(name="fotulix", parse_config=FotulixConfig.from_dict, model_spec=fotulix_model_spec)
register_architecture(["fotulix"], FOTULIX)
