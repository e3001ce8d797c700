"""The Dozotar decoder as a registry entry: configuration -> model spec.

A plain token embedding; layers in the order config.json lists them, each sublayer reading the residual stream itself
and its OUTPUT normed before it is added (the `output_norm` arrangement: x <- x + norm1(mixer(x)), x <- x +
norm2(ff(x))), every norm's weight one number; three kinds of mixer, grouped-query attention with a bias by the
distance's bucket inside chunks of positions (`attention`), linear attention with fixed decays (`retention`) and a
state-space recurrence (`mamba2`); a dense feed-forward gated by gelu, or routed experts with a gated shared one, or
none; a last RMS norm and a head of its own.  Nothing here computes: the spec names registered parts and hands them the
numbers of config.json.

Tensor names: `embed`, `head`, `final.norm`, and per layer i `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*` (a projection's norm
weight, convolution and bias with `.norm`, `.conv` and `.b` added to its name), `l<i>.mlp.gate|up|down`, or
`l<i>.mlp.router`, `l<i>.mlp.e<j>.gate|up|down`, `l<i>.mlp.shared.gate|up|down|sg`.
"""
from __future__ import annotations

from ..config.dozotar_config import (BucketAttentionConfig, DenseConfig, DozotarConfig, GroupedExpertsConfig, RetentionConfig,
                                     StateSpaceConfig)
from ..config.registry import ArchitectureFamily, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry

WEIGHT_SUM_EPS = 1e-20       # added to the sum of the chosen experts' scores that their weights are divided by


def _mixer_spec(cfg: DozotarConfig, m) -> PartSpec:
    if isinstance(m, BucketAttentionConfig):
        return PartSpec("distance_bias_attention", {
            "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
            "value_dim": m.vdim, "scale": m.scale, "bias": "buckets", "bias_far": m.bias_max, "block": m.mask_size,
            "conv_taps": m.conv, "qk_norm_eps": cfg.norm_eps})
    if isinstance(m, RetentionConfig):
        rope = None
        if m.rot_dims:
            rope = PartSpec("rope", {"head_dim": m.dim, "rotary_dim": m.rot_dims, "theta": m.rot_base, "scaling": None,
                                     "layout": "half"})
        return PartSpec("retention", {
            "hidden_size": cfg.width, "num_heads": m.heads, "key_dim": m.dim, "value_dim": m.vdim, "decay": list(m.decay),
            "k_scale": m.dim ** -0.5, "position": rope, "norm_eps": cfg.norm_eps})
    if isinstance(m, StateSpaceConfig):
        return PartSpec("mamba2", {
            "hidden_size": cfg.width, "num_heads": m.heads, "value_dim": m.vdim, "state_dim": m.state, "groups": m.groups,
            "conv_taps": m.conv, "norm_groups": m.norm_groups, "norm_eps": cfg.norm_eps})
    raise TypeError(f"no mixer for {type(m).__name__}")


def _ffn_spec(cfg: DozotarConfig, f) -> PartSpec:
    if isinstance(f, DenseConfig):
        return PartSpec("swiglu", {"hidden_size": cfg.width, "intermediate_size": f.ff, "activation": "gelu_tanh",
                                   "output": "float32", "gate_name": "gate", "up_name": "up", "down_name": "down"})
    if isinstance(f, GroupedExpertsConfig):
        return PartSpec("routed_experts", {
            "hidden_size": cfg.width, "expert_ff": f.ff, "experts": f.experts, "top": f.top, "score": "softmax",
            "groups_count": f.groups_count, "groups_keep": f.groups_keep, "group_score": "max", "renormalize": True,
            "renormalize_eps": WEIGHT_SUM_EPS, "shared_ff": f.shared_ff, "shared_gate": bool(f.shared_ff), "output": "float32"})
    raise TypeError(f"no feed-forward for {type(f).__name__}")


def dozotar_model_spec(cfg: DozotarConfig) -> ModelSpec:
    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": name, "scalar": True})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        names = {"mixer": p + "mix.", "post_mixer_norm": p}
        extra = {"post_mixer_norm": norm("norm1")}
        ffn = None
        if layer.mlp is not None:
            ffn = _ffn_spec(cfg, layer.mlp)
            extra["post_ffn_norm"] = norm("norm2")
            names.update({"ffn": p + "mlp.", "post_ffn_norm": p})
        layers.append(LayerSpec(mixer=_mixer_spec(cfg, layer.mixer), ffn=ffn, names=names, arrangement="output_norm",
                                extra_norms=extra))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab, layers=tuple(layers),
        run_order=tuple(RunEntry(i) for i in range(len(layers))),
        final_norm=norm(""), embed_name="embed", final_norm_name="final.norm", head_name="head", tie_head=False,
        eos_token_ids=cfg.eos_token_ids,
        embed=PartSpec("scaled_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "scale": 1.0, "weight_name": ""}),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight_name": ""}))


DOZOTAR = ArchitectureFamily(name="dozotar", parse_config=DozotarConfig.from_dict, model_spec=dozotar_model_spec)
register_architecture(["dozotar"], DOZOTAR)
