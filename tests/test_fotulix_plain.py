"""The plain Fotulix model against closed forms and hand-made cases, and what the package derives from a
config.json without a GPU: the typed configuration, the declared tensors, the cache layout, the tables by position,
configuration errors, the random-weights mode."""
import json
import math

import pytest
import torch

import plain_fotulix as P
from fotulix_helpers import CONFIGS, REL_ROWS, tensor_shapes

F64 = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


# ------------------------------------------------------------------------ the plain model
def test_rotation_by_hand():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0, 7.0]]], dtype=F64).repeat(3, 1, 1)      # [T=3, 1, 6], two pairs
    y = P.rotate_pairs(x, [1.0, 0.1], 2.0)
    assert torch.equal(y[0, 0], torch.tensor([2.0, 0.0, 0.0, 4.0, 5.0, 7.0], dtype=F64))  # the magnitude is on pairs alone
    for p in (1, 2):
        want = [2 * math.cos(p), 2 * math.sin(p), -4 * math.sin(0.1 * p), 4 * math.cos(0.1 * p), 5.0, 7.0]
        assert torch.allclose(y[p, 0], torch.tensor(want, dtype=F64))


def test_frequency_bands_by_hand():
    """Wavelengths 2 pi, 20 pi, 200 pi, 2000 pi over an original length of 400: below 400/4 kept, above 400/1 divided, the
    one of 200 pi = 628 divided too; between them the blend."""
    rot = {"dims": 8, "base": 10000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 400.0}}
    f = P.banded_frequencies(rot)
    assert f[:2] == [1.0, pytest.approx(0.1)] and f[2:] == [pytest.approx(0.01 / 8), pytest.approx(0.001 / 8)]
    rot["scaling"]["original"] = 1000.0                                               # 628 lies between 250 and 1000
    s = (1000.0 / (200 * math.pi) - 1.0) / 3.0
    assert P.banded_frequencies(rot)[2] == pytest.approx((1 - s) * 0.01 / 8 + s * 0.01)
    assert P.banded_frequencies({"dims": 4, "base": 100.0}) == [1.0, pytest.approx(0.1)]


def test_yarn_ramp_by_hand():
    """Sixteen channels, base 10000: pair(t) = 16 ln(1024 / (2 pi t)) / (2 ln 10000) is 1.4 for 32 turns and 4.4 for one:
    the ramp runs from pair 1 to pair 5."""
    rot = {"dims": 16, "base": 10000.0, "scaling": {"factor": 4.0, "original": 1024, "fast": 32.0, "slow": 1.0}}
    f, mag = P.yarn_frequencies(rot)
    plain = P.frequencies(rot)
    ratio = [a / b for a, b in zip(f, plain)]
    want = [1.0, 1.0, 0.75 + 0.25 / 4, 0.5 + 0.5 / 4, 0.25 + 0.75 / 4, 0.25, 0.25, 0.25]
    assert ratio == [pytest.approx(w) for w in want] and mag == pytest.approx(1.0 + 0.1 * math.log(4.0))
    assert P.yarn_frequencies({"dims": 16, "base": 10000.0}) == (plain, 1.0)


def test_query_temperature_by_hand():
    t = P.query_temperature(12, 0.5, 4)
    assert t[:3].tolist() == [1.0] * 3                                                # (p + 1) / 4 < 1
    assert t[3:7].tolist() == [pytest.approx(1 + 0.5 * math.log(2))] * 4
    assert t[7:11].tolist() == [pytest.approx(1 + 0.5 * math.log(3))] * 4 and t[11] == pytest.approx(1 + 0.5 * math.log(4))


def test_windows():
    m = P.visible(8, 3)
    assert m[5].tolist() == [False, False, False, True, True, True, False, False] and m[1].tolist() == [True, True] + [False] * 6
    assert P.visible(4, None)[3].tolist() == [True] * 4 and P.visible(3, 1)[2].tolist() == [False, False, True]


def test_distance_buckets_by_hand():
    got = [P.distance_bucket(n, 8, 64.0) for n in (0, 1, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 65, 5000)]
    assert got == [0, 1, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7, 7]


def test_a_sink_is_a_term_without_a_value():
    s = torch.log(torch.tensor([[[2.0, 99.0], [3.0, 5.0]]], dtype=F64))
    p = P.softmax_with_sink(s, P.visible(2, None), torch.log(torch.tensor([2.0], dtype=F64)))
    assert torch.allclose(p[0], torch.tensor([[0.5, 0.0], [0.3, 0.5]], dtype=F64))


def test_bigram_rows_by_hand():
    assert P.bigram_rows([4, 7, 7, 0], 10, 3, 13) == [13, (40 + 21) % 13, (70 + 21) % 13, 70 % 13]


def test_attention_scores_are_the_bias_alone_with_zero_queries():
    T, H, vd = 9, 2, 3
    table, v = rnd(4, H, seed=3), rnd(T, 1, vd, seed=2)
    q, k = torch.zeros(T, H, 5, dtype=F64), rnd(T, 1, 5, seed=1)
    bias = P.bias_by_distance(table, 6.0, T)
    out = P.grouped_attention(q, k, v, 0.7, bias=bias)
    for t in (0, 4, 8):
        for h in range(H):
            e = torch.exp(torch.tensor([float(table[P.distance_bucket(t - j, 4, 6.0), h]) for j in range(t + 1)], dtype=F64))
            assert torch.allclose(out[t, h], (e[:, None] * v[: t + 1, 0]).sum(0) / e.sum())
    assert torch.allclose(P.grouped_attention(q, k, v, 50.0, bias=bias), out)          # `scale` leaves the bias alone


def test_latent_layer_that_reads_anothers_rows():
    """With the owner's W_uk, W_uv and queries a reader is the owner; the rows are taken as they are."""
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 4, "kv_rank": 5, "scale": 0.3, "rot": {"dims": 2, "base": 10.0}, "mask": {"size": 3}}
    h = rnd(7, 6)
    w = {"q": rnd(10, 6, seed=1), "dkv": rnd(7, 6, seed=2), "dkv.norm": rnd(5, seed=3), "uk": rnd(6, 5, seed=4),
         "uv": rnd(8, 5, seed=5), "g": rnd(2, 6, seed=6), "o": rnd(6, 8, seed=7)}
    own = P.latent_attention(h, w, m, 1e-4)
    rows = P.latent_rows(h, w, m, 1e-4)
    assert torch.equal(P.latent_attention(h, {k: v for k, v in w.items() if not k.startswith("dkv")}, m, 1e-4, rows), own)
    # the first token: one key, so the heads' outputs are their values
    v = (rows[0][0] @ w["uv"].T).reshape(2, 4) * torch.sigmoid(h[0] @ w["g"].T)[:, None]
    assert torch.allclose(own[0], v.reshape(-1) @ w["o"].T)


def test_layer_written_out():
    """A model of one rotated layer of one token: its attention is v / (1 + exp(sink - score)), then the feed-forward, then
    the input by token, each behind its norm and with the residual's factor."""
    cfg = {"width": 4, "vocab": 7, "norm": {"eps": 1e-3}, "residual_mult": 0.6, "token_side": {"dim": 2},
           "embedding": {"scale": 2.0, "bigram": {"buckets": 3, "mul_prev": 1, "mul_cur": 2}}, "layers": [
        {"type": "attention_2", "mlp": {"kind": "dense", "ff": 3}, "mixer": {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.7}}]}
    shapes = {"embed": (7, 4), "bigram": (4, 4), "side.embed": (7, 2), "head": (7, 4), "final.norm": (4,), "l0.mix.q": (2, 4),
              "l0.mix.k": (2, 4), "l0.mix.v": (2, 4), "l0.mix.g": (1, 4), "l0.mix.o": (4, 2), "l0.mix.sink": (1,), "l0.mlp.gate": (3, 4),
              "l0.mlp.up": (3, 4), "l0.mlp.down": (4, 3), "l0.side.gate": (2, 4), "l0.side.proj": (4, 2), "l0.side.norm": (4,),
              "l0.norm1": (4,), "l0.norm1b": (4,), "l0.norm2": (4,), "l0.norm2b": (4,)}
    w = {n: rnd(*s, seed=i) for i, (n, s) in enumerate(shapes.items())}
    n = lambda y: y / torch.sqrt((y * y).mean() + 1e-3)
    x = 2.0 * w["embed"][5] + w["bigram"][3]
    h = n(x) * (1 + w["l0.norm1"])
    score = 0.7 * (w["l0.mix.q"] @ h) @ (w["l0.mix.k"] @ h)
    o = (w["l0.mix.v"] @ h) / (1 + torch.exp(w["l0.mix.sink"] - score)) / (1 + torch.exp(-w["l0.mix.g"] @ h))
    x = x + 0.6 * n(w["l0.mix.o"] @ o) * (1 + w["l0.norm1b"])
    h = n(x) * (1 + w["l0.norm2"])
    a = w["l0.mlp.gate"] @ h
    x = x + 0.6 * n(w["l0.mlp.down"] @ (a / (1 + torch.exp(-a)) * (w["l0.mlp.up"] @ h))) * (1 + w["l0.norm2b"])
    z = w["l0.side.gate"] @ x
    g = 0.5 * z * (1 + torch.tanh((2 / math.pi) ** 0.5 * (z + 0.044715 * z ** 3))) * w["side.embed"][5]
    x = x + 0.6 * n(w["l0.side.proj"] @ g) * w["l0.side.norm"]
    assert torch.allclose(P.forward(cfg, w, [5])[0], w["head"] @ (n(x) * (1 + w["final.norm"])))


# --------------------------------------------------------------------- tables the package makes
@pytest.mark.parametrize("dims,base,yarn", [(24, 70000.0, (6.0, 700, 24.0, 1.5)), (8, 3000.0, (3.0, 64, 8.0, 0.5)), (4, 40.0, (5.0, 30, 2.0, 1.0)),
                                            (64, 10000.0, (40.0, 4096, 32.0, 1.0)), (2, 10.0, (2.0, 16, 1.0, 1.0)), (12, 100.0, None)])
def test_yarn_tables(dims, base, yarn):
    from rustinfer_b200.parts.rope import RotaryEncoding
    rot = {"dims": dims, "base": base}
    scaling = None
    if yarn:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
        scaling = {"rope_type": "yarn", "factor": yarn[0], "original_max_position_embeddings": yarn[1], "beta_fast": yarn[2],
                   "beta_slow": yarn[3]}
    c, s = RotaryEncoding({"head_dim": dims, "rotary_dim": dims, "theta": base, "scaling": scaling}).tables(300)
    freq, mag = P.yarn_frequencies(rot)
    ang = torch.arange(300, dtype=F64)[:, None] * torch.tensor(freq, dtype=F64)
    assert torch.allclose(c, torch.cos(ang) * mag, atol=1e-12) and torch.allclose(s, torch.sin(ang) * mag, atol=1e-12)


@pytest.mark.parametrize("dims,base,bands", [(48, 30000.0, (6.0, 1.5, 5.0, 1500)), (8, 500.0, (4.0, 1.0, 4.0, 48)), (40, 70.0, (2.0, 2.0, 3.0, 20))])
def test_banded_tables(dims, base, bands):
    from rustinfer_b200.config.fotulix_config import BandScaling
    from rustinfer_b200.parts.rope import RotaryEncoding
    scaling = dict(zip(("factor", "low", "high", "original"), bands))
    c, s = RotaryEncoding({"head_dim": dims, "theta": base, "scaling": BandScaling.from_dict(scaling).rope_scaling()}).tables(100)
    ang = torch.arange(100, dtype=F64)[:, None] * torch.tensor(P.banded_frequencies({"dims": dims, "base": base, "scaling": scaling}), dtype=F64)
    assert torch.allclose(c, torch.cos(ang), atol=1e-12) and torch.allclose(s, torch.sin(ang), atol=1e-12)


@pytest.mark.parametrize("coef,every", [(0.6, 200), (1.5, 3), (0.0, 7), (-0.2, 1), (0.3, 2.5)])
def test_query_temperature_table(coef, every):
    from rustinfer_b200.parts.rope import QueryTemperature
    assert torch.allclose(QueryTemperature({"coef": coef, "every": every}).table(700), P.query_temperature(700, coef, every), atol=1e-14)


# --------------------------------------------------------------------- configuration, registry
def test_registry_and_declared_tensors():
    import rustinfer_b200  # noqa: F401
    from rustinfer_b200.config.registry import resolve_architecture
    from rustinfer_b200.models.decoder import Decoder
    for name, cfg in CONFIGS.items():
        fam = resolve_architecture(cfg)
        assert fam.name == "fotulix"
        typed = fam.parse_config(cfg, None)
        assert typed.to_dict() == cfg
        spec = fam.model_spec(typed)
        spec.validate()
        decls = Decoder(spec).param_decls()
        want = {n: ((-1,) + s[1:] if n.endswith(".rel") else s) for n, s in tensor_shapes(name).items()}
        assert {n: tuple(d.shape) for n, d in decls.items()} == want
        assert [e.cache_of for e in spec.run_order] == [l["mixer"].get("kv_from") for l in cfg["layers"]]


def test_cache_layout_of_mixed_layers():
    """Attention keeps every key, a latent layer as many rows as the widest of its readers sees, the stem one token."""
    import rustinfer_b200  # noqa: F401
    from rustinfer_b200.cache.manager import CacheLayout
    from rustinfer_b200.config.registry import resolve_architecture
    from rustinfer_b200.models.decoder import Decoder
    from rustinfer_b200.parts.base import FixedState, PagedKV

    def layout(name):
        fam = resolve_architecture(CONFIGS[name])
        needs = Decoder(fam.model_spec(fam.parse_config(CONFIGS[name], None))).cache_needs()
        return [n for _, n, _ in needs], CacheLayout.from_needs(needs)
    needs, lay = layout("A")
    row = PagedKV(1, 32, 37, value_dim=24, value_in_key=True)
    assert needs == [PagedKV(2, 24, None, value_dim=40), row, PagedKV(1, 24, None, value_dim=8), row,
                     PagedKV(3, 16, None, value_dim=24), FixedState((1,), "int32")]
    assert lay.entry_cache[3] == lay.entry_cache[1] and lay.entry_writes == [True, True, True, False, True, True]
    assert len(lay.paged_groups()) == 4 and row.first_key_kept(100) == 64
    needs, lay = layout("B")                                                          # no pairs of tokens: the stem keeps nothing
    assert len(needs) == 5 and needs[0].window == 16 and lay.entry_cache[1] == lay.entry_cache[4] == lay.entry_cache[0]
    assert layout("C")[0][2].window is None                                           # a reader sees every row


@pytest.mark.parametrize("change,needle", [
    (lambda c: c["layers"][0].__setitem__("type", "gla"), "mixer type"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("bias_max", 0), "bias_max"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].__setitem__("every", 0), "q_temp.every"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].pop("coef"), "coef"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 6), "rot.dims = rot_dim"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("rot_dim", 7), "even rot_dim"),
    (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][2]["mixer"]["rot"].__setitem__("dims", 26), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"].__setitem__("dims", 7), "even count"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].__setitem__("low", 5.0), "low < high"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 4), "does not run before"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 2), "caches none"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_rank", 20), "differ in kv_rank"),
    (lambda c: c["layers"][3]["mixer"]["rot"].__setitem__("base", 20.0), "differ in kv_rank"),
    (lambda c: c["embedding"]["bigram"].__setitem__("buckets", 0), "buckets"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda c: c["token_side"].__setitem__("dim", 0), "token_side"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_configuration_errors(change, needle):
    from rustinfer_b200.config.fotulix_config import FotulixConfig
    from rustinfer_b200.config.model_config import ConfigError
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    change(cfg)
    with pytest.raises(ConfigError, match=needle):
        FotulixConfig.from_dict(cfg)


def test_what_config_leaves_out_does_not_exist():
    from rustinfer_b200.config.fotulix_config import FotulixConfig
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    for key in ("kv_heads", "vdim", "q_temp"):
        cfg["layers"][0]["mixer"].pop(key)
    cfg["layers"] = cfg["layers"][:3]
    cfg["layers"][1]["mixer"].pop("mask")
    cfg["layers"][1]["mixer"]["rot"].pop("scaling")
    cfg["layers"][2]["mixer"].pop("rot")
    for key in ("embedding", "residual_mult", "token_side"):
        cfg.pop(key)
    c = FotulixConfig.from_dict(cfg)
    a, l, r = (x.mixer for x in c.layers)
    assert (a.kv_heads, a.vdim, a.temp_every) == (4, 24, None) and l.mask_size is None and l.rot.scaling is None and r.rot is None
    assert (c.embedding_scale, c.bigram, c.residual_mult, c.side_dim) == (1.0, None, 1.0, None) and c.layers[1].mlp is None
    cfg["layers"][0]["mixer"]["taper"] = 3
    with pytest.warns(UserWarning, match="taper"):
        FotulixConfig.from_dict(cfg)


def test_random_weights_mode(tmp_path):
    import rustinfer_b200  # noqa: F401
    from rustinfer_b200.weights.random_init import FREE_SIZE, write_random_model
    folder = write_random_model(str(tmp_path / "m"), CONFIGS["C"], seed=3, norm_std=0.1)
    cfg, w = P.read_model_folder(folder)
    want = {n: ((FREE_SIZE,) + s[1:] if n.endswith(".rel") else s) for n, s in tensor_shapes("C").items()}
    assert {n: tuple(t.shape) for n, t in w.items()} == want and REL_ROWS[("C", 1)] == 6
    logits = P.forward(cfg, w, [1, 5, 9, 96])
    assert logits.shape == (4, 101) and bool(torch.isfinite(logits).all())
