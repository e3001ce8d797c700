"""The plain Dozotar model against closed forms and hand-made cases, and what the package derives from a
config.json without a GPU: the typed configuration, the declared tensors, the cache layout, the bias by distance,
configuration errors, the random-weights mode."""
import json
import math

import pytest
import torch

import plain_dozotar as P
from dozotar_helpers import CONFIGS, REL_ROWS, tensor_shapes

F64 = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


# ------------------------------------------------------------------------ the plain model
def test_rotation_by_hand():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0, 7.0]]], dtype=F64).repeat(3, 1, 1)      # [T=3, 1, 6], dims 4
    y = P.rotate_half(x, torch.arange(3), 4, 100.0)
    assert torch.equal(y[0], x[0])                                                       # position 0: no turn
    for p in (1, 2):
        a0, a1 = p * 1.0, p * 100.0 ** (-2.0 / 4)                                        # pairs (0, 2) and (1, 3)
        want = [math.cos(a0), -2.0 * math.sin(a1), math.sin(a0), 2.0 * math.cos(a1), 5.0, 7.0]
        assert torch.allclose(y[p, 0], torch.tensor(want, dtype=F64))


def test_chunks_are_counted_from_position_0():
    m = P.chunk_mask(8, 3)
    assert m[5].tolist() == [False, False, False, True, True, True, False, False]
    assert m[6].tolist() == [False] * 6 + [True, False]                                   # a chunk's first sees itself alone
    assert m[2].tolist() == [True] * 3 + [False] * 5
    assert P.chunk_mask(4, None)[3].tolist() == [True] * 4


def test_distance_buckets_by_hand():
    """8 rows, far 64: a row a distance up to 3, then 4 rows over ln(n/4)/ln(16): 4 .. 7 -> 4, 8 .. 15 -> 5,
    16 .. 31 -> 6, 32 and on -> 7."""
    got = [P.distance_bucket(n, 8, 64.0) for n in (0, 1, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 65, 5000)]
    assert got == [0, 1, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7, 7]
    assert [P.distance_bucket(n, 5, 30.0) for n in (0, 1, 2, 4, 5, 12, 13, 30, 400)] == [0, 1, 2, 2, 3, 3, 4, 4, 4]


def test_attention_scores_are_the_bias_alone_with_zero_queries():
    T, H, vd = 9, 2, 3
    table = rnd(4, H, seed=3)
    v = rnd(T, 1, vd, seed=2)
    q, k = torch.zeros(T, H, 5, dtype=F64), rnd(T, 1, 5, seed=1)
    out = P.biased_attention(q, k, v, 0.7, 5, table, 6.0)
    for t in (4, 5, 8):
        lo = t // 5 * 5
        for h in range(H):
            e = torch.exp(torch.tensor([float(table[P.distance_bucket(t - j, 4, 6.0), h]) for j in range(lo, t + 1)], dtype=F64))
            assert torch.allclose(out[t, h], (e[:, None] * v[lo: t + 1, 0]).sum(0) / e.sum())
    # `scale` multiplies the product of query and key, not the bias
    assert torch.allclose(P.biased_attention(q, k, v, 50.0, 5, table, 6.0), out)


def test_causal_convolution_by_hand():
    x = torch.tensor([[1.0], [10.0], [100.0], [1000.0]], dtype=F64)
    w = torch.tensor([[3.0, 2.0, 1.0]], dtype=F64)                                       # last column: the current token
    assert P.causal_conv(x, w).flatten().tolist() == [1.0, 12.0, 123.0, 1230.0]
    assert P.causal_conv(x, w[:, 2:], torch.tensor([0.5], dtype=F64)).flatten().tolist() == [1.5, 10.5, 100.5, 1000.5]


def test_walk_is_a_decayed_sum():
    T, H, d, vd = 6, 2, 3, 4
    k, q, v = rnd(T, H, d), rnd(T, H, d, seed=1), rnd(T, H, vd, seed=2)
    a = torch.sigmoid(rnd(T, H, seed=3))
    o = P.state_walk(k, v, q, a)
    for t in (0, 3, 5):
        for h in range(H):
            want = sum(torch.prod(a[s + 1: t + 1, h]) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert torch.allclose(o[t, h], want)


def test_state_space_mixer_of_one_token():
    """The first token: x, B, C through the last tap and silu; y = (C . B) dt x + D x; gate, then the norm a part."""
    m = {"heads": 2, "vdim": 2, "state": 3, "groups": 1, "conv": 3, "norm_groups": 2}
    h = rnd(1, 5)
    w = {"in": rnd(4 + 10 + 2, 5, seed=1), "conv": rnd(10, 3, seed=2), "conv.b": rnd(10, seed=3), "dt_bias": rnd(2, seed=4),
         "A_log": rnd(2, seed=5), "D": rnd(2, seed=6), "norm": rnd(4, seed=7), "o": torch.eye(4, dtype=F64)}
    u = (h @ w["in"].T)[0]
    c = u[4:14] * w["conv"][:, 2] + w["conv.b"]
    c = c / (1 + torch.exp(-c))
    dt = torch.log1p(torch.exp(u[14:] + w["dt_bias"]))
    y = torch.stack([((c[4:7] @ c[7:10]) * dt[i] + w["D"][i]) * c[2 * i: 2 * i + 2] for i in range(2)]).flatten()
    g = y * u[:4] / (1 + torch.exp(-u[:4]))
    want = torch.cat([g[:2] / torch.sqrt((g[:2] ** 2).mean() + 1e-3), g[2:] / torch.sqrt((g[2:] ** 2).mean() + 1e-3)]) * w["norm"]
    assert torch.allclose(P.mamba2(h, w, m, 1e-3)[0], want)


def test_router_by_hand():
    z = torch.log(torch.tensor([[0.20, 0.18, 0.05, 0.30, 0.17, 0.10]], dtype=F64))
    ids, wts = P.route(z, 2)
    assert ids.tolist() == [[3, 0]] and torch.allclose(wts, torch.tensor([[0.6, 0.4]], dtype=F64))
    # three groups of two: their largest are 0.20, 0.30, 0.17; with two kept the last pair is out, not by its sum
    ids, wts = P.route(z, 3, {"count": 3, "keep": 2})
    assert ids.tolist() == [[3, 0, 1]] and torch.allclose(wts.sum(), torch.tensor(1.0, dtype=F64))
    ids, _ = P.route(z, 2, {"count": 3, "keep": 1})
    assert ids.tolist() == [[3, 2]]


def test_layer_norms_the_outputs_alone():
    """A model of one retention layer without a feed-forward, written out."""
    cfg = {"width": 4, "vocab": 7, "norm": {"eps": 1e-3}, "layers": [
        {"type": "retention", "mlp": None, "mixer": {"heads": 1, "dim": 2, "vdim": 2, "decay": [0.5]}}]}
    shapes = {"embed": (7, 4), "head": (7, 4), "final.norm": (), "l0.norm1": (), "l0.mix.q": (2, 4), "l0.mix.k": (2, 4),
              "l0.mix.v": (2, 4), "l0.mix.g": (2, 4), "l0.mix.o": (4, 2)}
    w = {n: rnd(*s, seed=i) for i, (n, s) in enumerate(shapes.items())}
    ids = [3, 0, 6]
    x = w["embed"][ids]
    q, k, v, g = (x @ w["l0.mix." + n].T for n in "qkvg")
    o = torch.stack([sum(0.5 ** (t - s) * (q[t] @ k[s]) * 2 ** -0.5 * v[s] for s in range(t + 1)) for t in range(3)])
    n = lambda y: y / torch.sqrt((y * y).mean(-1, keepdim=True) + 1e-3)
    y = (n(o) * g / (1 + torch.exp(-g))) @ w["l0.mix.o"].T
    x = x + n(y) * w["l0.norm1"]
    assert torch.allclose(P.forward(cfg, w, ids), n(x) * w["final.norm"] @ w["head"].T)


# --------------------------------------------------------------------- configuration, registry
@pytest.mark.parametrize("rows,far", [(16, 120.0), (8, 64.0), (5, 30.0), (32, 128.0), (2, 9.0), (1, 3.0), (9, 4.5), (12, 1000.0), (7, 2.0)])
def test_bias_by_distance(rows, far):
    from rustinfer_b200.parts.attention_variants import bucket_bias
    table = torch.arange(rows * 3, dtype=torch.float32).reshape(rows, 3)
    full = bucket_bias(table, far)
    assert full.shape[0] == 3 and full.dtype == torch.float32 and full.is_contiguous()
    for n in list(range(0, 300)) + [1000, 4096]:
        want = 0 if rows == 1 else rows - 1 if n >= rows // 2 and far <= rows // 2 else P.distance_bucket(n, rows, far)
        assert full[:, min(n, full.shape[1] - 1)].tolist() == table[want].tolist(), n
    short = bucket_bias(table, far, 10)
    assert short.shape[1] <= 10 and torch.equal(short, full[:, : short.shape[1]])


def test_registry_and_declared_tensors():
    import rustinfer_b200  # noqa: F401
    from rustinfer_b200.config.registry import resolve_architecture
    from rustinfer_b200.models.decoder import Decoder
    for name, cfg in CONFIGS.items():
        fam = resolve_architecture(cfg)
        assert fam.name == "dozotar"
        typed = fam.parse_config(cfg, None)
        assert typed.to_dict() == cfg
        spec = fam.model_spec(typed)
        decls = Decoder(spec).param_decls()
        want = {n: ((-1,) + s[1:] if n.endswith(".rel") else s) for n, s in tensor_shapes(name).items()}
        assert {n: tuple(d.shape) for n, d in decls.items()} == want
        assert [ls.arrangement for ls in spec.layers] == ["output_norm"] * len(cfg["layers"])


def test_cache_layout_of_mixed_layers():
    """Attention keeps the pages of the current chunk and its convolution's last inputs, retention a matrix a head, the
    state-space layer its convolution's inputs and a matrix a head."""
    import rustinfer_b200  # noqa: F401
    from rustinfer_b200.cache.manager import CacheLayout
    from rustinfer_b200.config.registry import resolve_architecture
    from rustinfer_b200.models.decoder import Decoder
    from rustinfer_b200.parts.base import FixedState, PagedKV
    fam = resolve_architecture(CONFIGS["A"])
    dec = Decoder(fam.model_spec(fam.parse_config(CONFIGS["A"], None)))
    needs = [n for _, n, _ in dec.cache_needs()]
    assert needs[0] == (PagedKV(2, 24, None, value_dim=40, block=20), FixedState((2, 4 * 24 + 2 * 24 + 2 * 40)))
    assert needs[1] == (FixedState((1, 6 * 20 + 2 * 3 * 24)), FixedState((6, 20, 32)))      # 24 rows in 8 lanes of 4
    assert needs[2] == FixedState((3, 12, 32))
    assert needs[0][0].first_key_kept(100) == 100 and needs[0][0].first_key_kept(99) == 80
    assert len(CacheLayout.from_needs(dec.cache_needs()).paged_groups()) == 1
    famc = resolve_architecture(CONFIGS["C"])
    decc = Decoder(famc.model_spec(famc.parse_config(CONFIGS["C"], None)))
    assert decc.cache_needs()[2][1][0] == FixedState((0, 5 * 7 + 2 * 5 * 9))                # one tap keeps nothing


@pytest.mark.parametrize("change,needle", [
    (lambda c: c["layers"][0].__setitem__("type", "gla"), "mixer type"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "relu"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("bias_max", 0), "bias_max"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("groups", 4), "multiple of groups"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("norm_groups", 7), "norm_groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].__setitem__("top", 9), "top <= experts"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].__setitem__("count", 3), "groups.count"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].__setitem__("keep", 1), "at least `top`"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("decay", [0.9, 0.8]), "decay"),
    (lambda c: c["layers"][2]["mixer"]["rot"].__setitem__("dims", 22), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"].__setitem__("dims", 7), "rot.dims"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_configuration_errors(change, needle):
    from rustinfer_b200.config.dozotar_config import DozotarConfig
    from rustinfer_b200.config.model_config import ConfigError
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    change(cfg)
    with pytest.raises(ConfigError, match=needle):
        DozotarConfig.from_dict(cfg)


def test_what_config_leaves_out_does_not_exist():
    from rustinfer_b200.config.dozotar_config import DozotarConfig
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    for key in ("kv_heads", "vdim", "mask"):
        cfg["layers"][0]["mixer"].pop(key)
    cfg["layers"][1]["mlp"].pop("shared")
    cfg["layers"][1]["mlp"]["router"].pop("groups")
    cfg["layers"][2]["mixer"].pop("rot")
    c = DozotarConfig.from_dict(cfg)
    a, e = c.layers[0].mixer, c.layers[1].mlp
    assert (a.kv_heads, a.vdim, a.mask_size) == (4, 24, None)
    assert (e.shared_ff, e.groups_count) == (None, 0) and c.layers[2].mixer.rot_dims == 0 and c.layers[2].mlp is None
    cfg["layers"][0]["mixer"]["taper"] = 3
    with pytest.warns(UserWarning, match="taper"):
        DozotarConfig.from_dict(cfg)


def test_random_weights_mode(tmp_path):
    import rustinfer_b200  # noqa: F401
    from rustinfer_b200.weights.random_init import FREE_SIZE, write_random_model
    folder = write_random_model(str(tmp_path / "m"), CONFIGS["C"], seed=3, norm_std=0.1)
    cfg, w = P.read_model_folder(folder)
    want = {n: ((FREE_SIZE,) + s[1:] if n.endswith(".rel") else s) for n, s in tensor_shapes("C").items()}
    assert {n: tuple(t.shape) for n, t in w.items()} == want and REL_ROWS[("C", 1)] == 5
    assert cfg["layers"][2]["mlp"] is None and abs(float(w["l0.norm1"]) - 1.0) < 0.5
    logits = P.forward(cfg, w, [1, 5, 9, 96])
    assert logits.shape == (4, 97) and bool(torch.isfinite(logits).all())
