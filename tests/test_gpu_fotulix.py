"""The Fotulix family on the GPU against the plain implementation: every new kernel alone, every mixer alone with a key made
to stand out at the edges of its window, then the engine under every way of cutting the work (whole prompts, a decoded tail,
portions down to two tokens, mixed batches with pages and state slots used again), in true 32-bit and in bfloat16, on small
configurations that differ in every size; greedy generation through `Engine`; the trace replay command and the command line."""
import json
import os
import subprocess

import pytest
import torch

import plain_fotulix as P
from fotulix_helpers import CONFIGS, MixerRig, Plain, make_sharp_model
from helpers import random_ids, rel_err

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"
F64 = torch.float64
BF = torch.bfloat16
# max |engine - plain| / max |plain| over the compared logits.  fp32 sums a few hundred products per output
# against float64, and every sublayer's output is divided by its own root mean square before it is added (a small
# output's rounding grows with it); in bfloat16 projections and activations are rounded to 8 bits.
TOL = {"float32": 2e-5, "bfloat16": 6e-2}
DTYPES = ["float32", "bfloat16"]
NAMES = sorted(CONFIGS)


def K():
    from rustinfer_b200.ops import kernels
    return kernels


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float32) * scale


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def pieces(T, cuts):
    out, at = [], 0
    while at < T:
        for c in cuts:
            if at >= T:
                break
            out.append((at, min(T, at + c)))
            at = out[-1][1]
    return out


# ================================================================================= kernels alone
@pytest.mark.parametrize("d,vocab,buckets,mp,mc", [(96, 211, 61, 17, 5), (83, 40, 1, 3, 2), (1032, 100, 7919, 2147483647, 1099511627791),
                                                   (64, 128000, 65521, 40503, 9973), (20, 50, 1000, 0, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_embedding_of_token_pairs_in_pieces(d, vocab, buckets, mp, mc, dtype):
    """Two requests side by side in slots of their own, in pieces of 1, 2 and many tokens: the pair across a piece's border
    comes from the slot, a request's first token has the table's last row, and no other slot is touched."""
    T = [61, 34]
    ids = [random_ids(n, vocab, 5 + i) for i, n in enumerate(T)]
    ids[0][3], ids[0][7] = vocab - 1, vocab - 1
    table, pairs = rnd(vocab, d, seed=1).to(dtype), rnd(buckets + 1, d, seed=2).to(dtype)
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    state = torch.full((4, 1), 77777777, dtype=torch.int32, device=DEV)
    state[[1, 3]] = 0
    got = [torch.empty(n, d) for n in T]
    cut = [pieces(T[0], [1, 2, 1, 30, 3]), pieces(T[1], [2, 1, 1, 13])]
    for step in range(max(len(c) for c in cut)):
        toks, pos, slots, cu, parts = [], [], [], [0], []
        for r, slot in ((0, 3), (1, 1)):
            if step < len(cut[r]):
                a, b = cut[r][step]
                toks += ids[r][a:b]; pos += list(range(a, b)); slots.append(slot); cu.append(cu[-1] + b - a); parts.append((r, a, b))
        out = torch.empty(len(toks), d, device=DEV)
        K().embed_pairs(i32(toks), i32(pos), i32(cu), i32(slots), len(slots), state, table.to(DEV), 2.5, pairs.to(DEV), mp, mc, out)
        for (r, a, b), lo in zip(parts, cu):
            got[r][a:b] = out[lo: lo + b - a].cpu()
            assert int(state[[3, 1][r]]) == ids[r][b - 1]
    for r in range(2):
        assert rel_err(got[r], P.embedding(cfg, {"embed": table, "bigram": pairs}, ids[r])) < 1e-6
    assert state[[0, 2]].flatten().tolist() == [77777777] * 2


@pytest.mark.parametrize("T,n,columns,column,vocab", [(1, 12, 60, 12, 211), (70, 7, 28, 21, 101), (300, 256, 1024, 512, 500), (5, 1, 1, 0, 9)])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_gate_by_token(T, n, columns, column, vocab, dtype):
    z, table, ids = rnd(T, n + 3, seed=1, scale=2.0), rnd(vocab, columns, seed=2).to(dtype), random_ids(T, vocab, 3)
    out = torch.empty(T, n, dtype=dtype, device=DEV)
    K().token_gate(z.to(DEV)[:, 3:], i32(ids), table.to(DEV), column, out)
    want = P.gelu_tanh(z[:, 3:].to(F64)) * table.to(F64)[ids][:, column: column + n]
    assert rel_err(out, want) < (2e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("T,d,dim,vocab,layers", [(1, 96, 12, 211, 3), (70, 92, 7, 101, 4), (600, 256, 64, 90, 2), (9, 64, 20, 97, 3)])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_input_by_token(T, d, dim, vocab, layers, dtype):
    """The part against the plain statement, its columns of the shared table by the layer's number."""
    import rustinfer_b200.models.decoder  # noqa: F401  (registers the built-in parts)
    from types import SimpleNamespace
    from rustinfer_b200.parts.base import BuildContext, FEED_FORWARDS
    from rustinfer_b200.parts.spec import PartSpec
    ids, x = random_ids(T, vocab, 3), rnd(T, d, seed=5).to(dtype)
    table = rnd(vocab, dim * layers, seed=6).to(dtype)
    for i in (0, layers - 1):
        part = FEED_FORWARDS.build(PartSpec("token_input", {
            "hidden_size": d, "vocab_size": vocab, "dim": dim, "table_columns": dim * layers, "column": i * dim,
            "table_name": "t", "gate_name": "g", "proj_name": "p"}))
        part.prepare(BuildContext(torch.device(DEV), dtype, 64, 16))
        w = {"gate": rnd(dim, d, seed=7 + i, scale=0.2).to(dtype), "proj": rnd(d, dim, seed=8 + i, scale=0.2).to(dtype),
             "norm": torch.ones(d)}
        part.load({"t": table.to(DEV), "g": w["gate"].to(DEV), "p": w["proj"].to(DEV)})
        got = part.forward(x.to(DEV), SimpleNamespace(token_ids=i32(ids + [0])))
        e = table.to(F64)[ids][:, i * dim: (i + 1) * dim]
        want = (P.gelu_tanh(x.to(F64) @ w["gate"].to(F64).T) * e) @ w["proj"].to(F64).T
        assert got.dtype == torch.float32 and rel_err(got, want) < (1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 24, 40, 0), (3, 3, 23, 9, 0), (4, 1, 24, 8, 8), (8, 1, 16, 32, 16)])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_queries_with_bias_temperature_and_rotation(H, G, dk, dv, rot, dtype):
    from rustinfer_b200.parts.rope import QueryTemperature, RotaryEncoding
    page, pos = 4, [0, 1, 2, 30, 31, 32, 4000, 77, 4095]
    T, cols = len(pos), H * dk + G * dk + G * dv
    x, bias = rnd(T, cols + 4, seed=1), rnd(cols, seed=2)
    factor = QueryTemperature({"coef": 0.7, "every": 16}).table(4096)
    c, s = RotaryEncoding({"head_dim": dk, "rotary_dim": rot or 2, "theta": 300.0, "layout": "interleaved"}).tables(4096)
    shape = (6, 2, G, page, dk) if dk == dv else (6, page * G * (dk + dv))
    cache = torch.full(shape, 33.0, dtype=dtype, device=DEV)
    place = torch.randperm(24, generator=torch.Generator().manual_seed(2))[:T]
    q = torch.empty(T, H * dk, dtype=dtype, device=DEV)
    K().qkv_prepare(x.to(DEV)[:, :cols], bias.to(DEV), None, None, 0, 0.0, i32(pos), c.float().to(DEV) if rot else None,
                    s.float().to(DEV) if rot else None, rot, True, i32(place.tolist()), cache, q, H, G, dk, dv, True,
                    q_scale=factor.float().to(DEV))
    y = (x[:, :cols] + bias).to(F64)

    def turned(v, heads):
        v = v.reshape(T, heads, dk).clone()
        if rot:
            cc, ss = c[pos][:, None], s[pos][:, None]
            a, b = v[..., 0:rot:2].clone(), v[..., 1:rot:2].clone()
            v[..., 0:rot:2], v[..., 1:rot:2] = a * cc - b * ss, b * cc + a * ss
        return v
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    assert rel_err(q, (turned(y[:, : H * dk], H) * factor[pos][:, None, None]).reshape(T, -1)) < tol
    kk, vv = turned(y[:, H * dk: H * dk + G * dk], G), y[:, H * dk + G * dk:].reshape(T, G, dv)
    flat = cache.reshape(-1, page * G * (dk + dv)).float().cpu()
    for t in range(T):
        pg, off = divmod(int(place[t]), page)
        assert rel_err(flat[pg][: G * page * dk].view(G, page, dk)[:, off], kk[t]) < 10 * tol
        assert rel_err(flat[pg][G * page * dk:].view(G, page, dv)[:, off], vv[t]) < 10 * tol


@pytest.mark.parametrize("H,d,r,rank", [(3, 16, 8, 24), (1, 5, 4, 20), (12, 16, 16, 80)])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_latent_queries_alone(H, d, r, rank, dtype):
    """A layer that reads another's rows prepares its queries and writes nothing."""
    T, kd = 9, rank + r
    pos = [0, 1, 5, 100, 2047, 8, 9, 10, 11]
    from rustinfer_b200.parts.rope import RotaryEncoding
    c, s = RotaryEncoding({"head_dim": r, "theta": 100.0, "scaling": {
        "rope_type": "yarn", "factor": 3.0, "original_max_position_embeddings": 64, "beta_fast": 4.0, "beta_slow": 1.0}}).tables(2048)
    x = rnd(T, H * (d + r) + 5, seed=1)
    qp = torch.empty(T, H * d, dtype=dtype, device=DEV)
    qf = torch.full((T, H * kd), 7.0, dtype=dtype, device=DEV)
    K().latent_prepare(x.to(DEV)[:, : H * (d + r)], None, 0.0, i32(pos), c.float().to(DEV), s.float().to(DEV), None, None, qp, qf, H, d, r,
                       rank)
    v = x[:, : H * (d + r)].to(F64).view(T, H, d + r)
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    assert rel_err(qp, v[..., :d].reshape(T, -1)) < tol
    a, b, cc, ss = v[..., d::2], v[..., d + 1:: 2], c[pos][:, None], s[pos][:, None]
    want = torch.stack([a * cc - b * ss, b * cc + a * ss], dim=-1).reshape(T, H, r)
    got = qf.view(T, H, kd).double().cpu()
    assert rel_err(got[..., rank:], want) < tol and bool((got[..., :rank] == 7.0).all())


@pytest.mark.parametrize("H,G,dk,dv,maps,vik", [(4, 2, 64, 64, 1, False), (8, 1, 16, 32, 1, False), (20, 1, 32, 16, 1, False), (6, 2, 48, 80, 1, False),
                                               (12, 2, 16, 48, 2, False), (3, 3, 128, 128, 1, False), (12, 1, 96, 80, 1, True), (70, 1, 32, 16, 1, True),
                                               (5, 1, 160, 128, 1, True), (40, 2, 16, 16, 1, False)])
@pytest.mark.parametrize("page", [8, 16, 12])
def test_single_tokens_on_the_tensor_cores(H, G, dk, dv, maps, vik, page):
    """The kernel whose warps share the keys of one entry: groups of 1 to 70 heads, maps, values inside the keys, every option
    of the scores, a gate; a far key and keys at the window's edges made to stand out; lengths of one key and more, in 1 to 7
    ranges of which some are empty; pages scrambled, the rest poisoned; other entries of the batch untouched."""
    lens = [1, 2, 33, 64, 257, 330]
    per = G * (maps * dk + (0 if vik else dv))
    blocks = -(-max(lens) // page)
    tab = (torch.randperm(len(lens) * blocks, generator=torch.Generator().manual_seed(5)) + 1).view(len(lens), blocks)
    keys = [torch.nn.functional.normalize(rnd(n, G * maps, dk, seed=10 + i), dim=-1) * 4.0 for i, n in enumerate(lens)]
    keys = [k.to(BF).float() for k in keys]
    vals = [k[:, :, :dv] if vik else rnd(n, G, dv, seed=30 + i).to(BF).float() for i, (n, k) in enumerate(zip(lens, keys))]
    cache = torch.full((len(lens) * blocks + 1, page * per), 1e4)
    for i, n in enumerate(lens):
        for t in range(n):
            row, off = cache[int(tab[i, t // page])], t % page
            row[: G * maps * page * dk].view(G * maps, page, dk)[:, off] = keys[i][t]
            if not vik:
                row[G * maps * page * dk:].view(G, page, dv)[:, off] = vals[i][t]
    plain = maps == 1 and dk == dv and not vik
    dev_cache = cache.to(BF).to(DEV)
    dev_cache = dev_cache.view(-1, 2, G, page, dk) if plain else dev_cache
    Q = 2 + len(lens)                                             # two more tokens in front, of an entry that is not single
    q, gate = rnd(Q, H, dk, seed=1), rnd(Q, H, seed=2)
    sink, slopes, bias = rnd(H, seed=3) + 1.0, torch.rand(H, generator=torch.Generator().manual_seed(4)) / 20, rnd(H, 40, seed=5) * 2
    per_head = H // (G * maps)
    kh_of = [(h // maps) // per_head * maps + h % maps for h in range(H)]
    vh_of = [(h // maps) // per_head for h in range(H)]
    for opt in ("plain", "window", "block", "bias", "bias_window", "slopes", "cap"):
        if vik and "bias" in opt:
            continue
        window = {"window": 37, "bias_window": 64}.get(opt)
        block = 50 if opt == "block" else None
        targets = [n - 1 if not window else max(0, n - window) for n in lens]       # the last key seen stands out
        if not window and not block:
            targets = [0] * len(lens)
        for i, (n, tg) in enumerate(zip(lens, targets)):
            for h in range(H):
                k = keys[i][tg, kh_of[h]]
                q[2 + i, h] = k * (0.75 + 0.02 * h / H)
        qr = q.to(BF).float()
        want = torch.empty(len(lens), H, dv, dtype=F64)
        for i, n in enumerate(lens):
            p = n - 1
            j = torch.arange(n)
            seen = (p - j < window) if window else torch.ones(n, dtype=torch.bool)
            if block:
                seen = seen & (j // block == p // block)
            for h in range(H):
                s = keys[i][:, kh_of[h]].to(F64) @ qr[2 + i, h].to(F64) * 0.9
                if opt == "cap":
                    s = 3.0 * torch.tanh(s / 3.0)
                if opt == "slopes":
                    s = s - slopes[h].to(F64) * (p - j)
                if "bias" in opt:
                    s = s + bias[h].to(F64)[(p - j).clamp(max=39)]
                w = P.softmax_with_sink(s[None, None], seen[None], sink[h].to(F64)[None] if opt != "block" else None)[0, 0]
                want[i, h] = (w @ vals[i][:, vh_of[h]].to(F64)) * torch.sigmoid(gate[2 + i, h].to(F64)) * 0.8
        table = i32([[0] * blocks] + tab.tolist())
        cu, kv = i32([0] + [2 + i for i in range(len(lens) + 1)]), i32([2] + lens)
        entries, zeros = i32([-1] + list(range(1, len(lens) + 1))), i32([0] * 8)
        for splits in (1, 2, 7):
            out = torch.full((Q, H * dv), 55.0, device=DEV)
            n = K().attention_rows_scratch_floats(entries.numel(), H, G, dv, maps, splits)
            part = torch.full((max(1, n),), float("nan"), device=DEV)
            K().attention_rows_single(qr.reshape(Q, -1).to(BF).to(DEV), out, dev_cache, table, cu, kv, entries, zeros, H, G, dk, 0.9, window, dv,
                                      sink=opt != "block", softcap=3.0 if opt == "cap" else None, sink_values=sink.to(DEV) if opt != "block" else None,
                                      maps=maps, value_in_key=vik, splits=splits, part=part, slopes=slopes.to(DEV) if opt == "slopes" else None,
                                      bias=bias.to(DEV) if "bias" in opt else None, block=block, gate=gate.to(DEV), gate_scale=0.8)
            assert float((out[2:].cpu().view(-1, H, dv).to(F64) - want).abs().max()) < 1e-4, (opt, splits)
            assert bool((out[:2] == 55.0).all())


# ================================================================================= mixers alone
def weights(shapes, seed):
    out = {}
    for i, (n, s) in enumerate(shapes.items()):
        t = rnd(*s, seed=seed + i, scale=s[-1] ** -0.5 if len(s) > 1 else 0.5)
        out[n] = (1.0 + t if n.endswith("norm") else t).to(BF).to(torch.float32)
    return out


CUTS = [[330], [270] + [1] * 60, [33, 1, 2, 2, 7, 16, 64, 5, 1, 1, 90, 2, 8, 98], [1] * 20 + [200] + [1, 2, 3, 4] * 11]


def planted(width, T, at, seed):
    """Inputs of one sequence: channel 0 is 1 everywhere (queries look along it), channel 1 is large at the token `at` alone
    (its key answers)."""
    h = rnd(T, width, seed=seed, scale=0.3)
    h[:, 0], h[:, 1] = 1.0, 0.0
    h[at, 1] = 8.0
    return h.to(BF).to(torch.float32)


def aim(w, key, H, d, rows, gain):
    """Let the queries' column 0 point along `key` [heads or 1, rows] in the first `rows` channels of every head's `d`."""
    q = w["q"].view(H, d, -1)
    k = key if key.shape[0] == H else key.repeat_interleave(H // key.shape[0], dim=0)
    q[:, :, 0] = 0.0
    q[:, :rows, 0] = gain * k / (k * k).sum(-1, keepdim=True)
    w["q"] = q.reshape(H * d, -1).to(BF).to(torch.float32)


def held(got, want, dtype, what):
    err = float((got - want).abs().max() / want.abs().max())
    assert err < (2e-5 if dtype == torch.float32 else 3e-2), (what, err)


@pytest.mark.parametrize("H,G,dim,vdim,rows,far,temp", [(4, 2, 24, 40, 8, 50.0, (0.4, 16)), (8, 1, 16, 32, 32, 200.0, None),
                                                         (2, 2, 32, 32, 16, 100.0, (0.1, 100)), (3, 3, 23, 9, 6, 9.0, (0.5, 3))])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_attention_with_bias_and_temperature_alone(H, G, dim, vdim, rows, far, temp, dtype):
    """A key at the sequence's start, at a page's edge and in its middle stands out for every later query, hundreds of tokens
    on: whole, in portions, and token by token; then random inputs, where bias and temperature alone tell keys apart."""
    from rustinfer_b200.parts.spec import PartSpec
    width, T = 40, 330
    m = {"heads": H, "kv_heads": G, "dim": dim, "vdim": vdim, "scale": dim ** -0.5, "bias_max": far}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    spec = PartSpec("gated_attention", {
        "hidden_size": width, "num_heads": H, "num_kv_heads": G, "head_dim": dim, "value_dim": vdim, "scale": m["scale"],
        "bias": "buckets", "bias_far": far, "proj_bias": True, "head_gate": True,
        "q_temperature": PartSpec("query_temperature", {"coef": temp[0], "every": temp[1]}) if temp else None})
    shapes = {"q": (H * dim, width), "k": (G * dim, width), "v": (G * vdim, width), "q.b": (H * dim,), "k.b": (G * dim,),
              "v.b": (G * vdim,), "g": (H, width), "o": (width, H * vdim), "rel": (rows, H)}
    for at in (0, 7, 40, None):
        w = weights(shapes, 10)
        w["rel"] = (w["rel"] * rows ** 0.5 * 1.5).to(BF).to(torch.float32)
        if at is None:
            h = rnd(T, width, seed=5).to(BF).to(torch.float32)
        else:
            h = planted(width, T, at, 6)
            aim(w, 8.0 * w["k"].view(G, dim, width)[:, :, 1], H, dim, dim, 14.0 / m["scale"])
        rig = MixerRig(spec, w, dtype)
        want = P.attention(h.to(F64), {k: v.to(F64) for k, v in w.items()}, m)
        if at is not None:                                                # the plant matters: without it the last query sees another
            other = h.clone()
            other[at, 1] = 0.0
            far_off = P.attention(other.to(F64), {k: v.to(F64) for k, v in w.items()}, m)
            assert float((far_off[-1] - want[-1]).abs().max() / want.abs().max()) > 0.2
        for cuts in CUTS:
            held(rig.run(h, cuts), want, dtype, (at, cuts[:3]))


@pytest.mark.parametrize("H,G,dim,vdim,rot,bands", [(4, 1, 24, 8, 8, (4.0, 1.0, 4.0, 48)), (6, 2, 32, 16, 24, None), (4, 2, 64, 48, 64, (2.0, 1.0, 2.0, 64)),
                                                    (1, 1, 40, 24, 40, None), (2, 1, 16, 24, 0, None), (16, 2, 16, 32, 16, None)])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_rotated_attention_with_a_sink_alone(H, G, dim, vdim, rot, bands, dtype):
    """A far key that stands out against the sink (where channels are left unrotated to plant it in), then random inputs with
    sinks that are negligible, level with the scores and dominant."""
    from rustinfer_b200.config.fotulix_config import BandScaling
    from rustinfer_b200.parts.spec import PartSpec
    width, T = 40, 330
    m = {"heads": H, "kv_heads": G, "dim": dim, "vdim": vdim, "scale": dim ** -0.5}
    rope = None
    if rot:
        m["rot"] = {"dims": rot, "base": 500.0}
        scaling = None
        if bands:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
            scaling = BandScaling.from_dict(m["rot"]["scaling"]).rope_scaling()
        rope = PartSpec("rope", {"head_dim": dim, "rotary_dim": rot, "theta": 500.0, "layout": "interleaved", "scaling": scaling})
    spec = PartSpec("gated_attention", {
        "hidden_size": width, "num_heads": H, "num_kv_heads": G, "head_dim": dim, "value_dim": vdim, "scale": m["scale"],
        "bias": "none", "position": rope, "sink": True, "head_gate": True})
    shapes = {"q": (H * dim, width), "k": (G * dim, width), "v": (G * vdim, width), "g": (H, width), "o": (width, H * vdim), "sink": (H,)}
    for at, sink in ((0, 5.0), (47, 5.0), (None, -20.0), (None, 1.0), (None, 12.0)):
        w = weights(shapes, 20)
        w["sink"] = torch.full((H,), sink) + torch.arange(H) / 8.0
        if at is None:
            h = rnd(T, width, seed=5).to(BF).to(torch.float32)
        elif rot == dim:
            continue
        else:
            h = planted(width, T, at, 6)
            key = 8.0 * w["k"].view(G, dim, width)[:, rot:, 1]
            k = w["k"].view(G, dim, width)
            k[:, :rot, 1] = 0.0
            q = w["q"].view(H, dim, width)
            q[:, :, 0] = 0.0
            kk = key.repeat_interleave(H // G, dim=0)
            q[:, rot:, 0] = 14.0 / m["scale"] * kk / (kk * kk).sum(-1, keepdim=True)
            w["q"], w["k"] = q.reshape(-1, width).to(BF).to(torch.float32), k.reshape(-1, width)
        rig = MixerRig(spec, w, dtype)
        want = P.attention_2(h.to(F64), {k: v.to(F64) for k, v in w.items()}, m)
        for cuts in CUTS:
            held(rig.run(h, cuts), want, dtype, (at, sink, cuts[:3]))


@pytest.mark.parametrize("H,dim,rd,vdim,rank,window,H2,dim2,vdim2,window2", [
    (3, 16, 8, 20, 24, 20, 5, 10, 12, 37), (8, 32, 16, 24, 32, 16, 2, 16, 32, 9), (12, 16, 16, 16, 80, 50, 8, 32, 48, 33),
    (1, 24, 4, 16, 20, 5, 2, 24, 16, 6), (2, 16, 8, 16, 24, 1, 4, 8, 8, None), (70, 8, 8, 8, 24, 64, 1, 8, 8, 65)])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_windowed_latent_attention_and_a_reader_alone(H, dim, rd, vdim, rank, window, H2, dim2, vdim2, window2, dtype):
    """One row stands out for every query: the last one that sees it and the first that does not, of the owner of the rows
    and of a layer that reads them with a window of its own, in prompt portions and for single tokens, with the row at a page's
    edges and in its middle; pages outside are poisoned."""
    from rustinfer_b200.parts.spec import PartSpec
    width, T, eps = 40, 330, 1e-4
    rot = {"dims": rd, "base": 300.0, "scaling": {"factor": 3.0, "original": 64, "fast": 4.0, "slow": 1.0}}
    scaling = {"rope_type": "yarn", "factor": 3.0, "original_max_position_embeddings": 64, "beta_fast": 4.0, "beta_slow": 1.0}
    keep = None if window2 is None else max(window, window2)

    def spec(heads, d, v, win, own):
        return PartSpec("latent_attention", {
            "hidden_size": width, "num_heads": heads, "head_dim": d, "rot_dim": rd, "value_dim": v, "kv_rank": rank, "scale": 0.25,
            "rot_base": 300.0, "rot_scaling": scaling, "norm_eps": eps, "gate": "head", "window": win, "cache_window": keep, "own_kv": own})

    def config(heads, d, v, win):
        m = {"heads": heads, "dim": d, "rot_dim": rd, "vdim": v, "kv_rank": rank, "scale": 0.25, "rot": rot}
        return dict(m, mask={"size": win}) if win else m

    def shapes(heads, d, v):
        return {"q": (heads * (d + rd), width), "uk": (heads * d, rank), "uv": (heads * v, rank), "g": (heads, width), "o": (width, heads * v)}
    m1, m2 = config(H, dim, vdim, window), config(H2, dim2, vdim2, window2)
    for at in (63, 64, 100, None):
        w1 = weights({**shapes(H, dim, vdim), "dkv": (rank + rd, width), "dkv.norm": (rank,)}, 30)
        w2 = weights(shapes(H2, dim2, vdim2), 50)
        w64 = lambda w: {k: v.to(F64) for k, v in w.items()}
        if at is None:
            h = rnd(T, width, seed=5).to(BF).to(torch.float32)
        else:
            h = planted(width, T, at, 6)
            c, _ = P.latent_rows(h.to(F64), w64(w1), m1, eps)
            for w, heads, d in ((w1, H, dim), (w2, H2, dim2)):
                key = (w["uk"].to(F64) @ c[at]).reshape(heads, d).float()
                aim(w, key, heads, d + rd, d, 14.0 / 0.25)
        rows = P.latent_rows(h.to(F64), w64(w1), m1, eps)
        want1 = P.latent_attention(h.to(F64), w64(w1), m1, eps, rows)
        want2 = P.latent_attention(h.to(F64), w64(w2), m2, eps, rows)
        if at is not None:                                   # one query further and the output is another one
            for want, win in ((want1, window), (want2, window2)):
                if win and win > 1:
                    a, b = want[at + win - 1], want[at + win]
                    assert float((a - b).abs().max() / b.abs().max()) > 0.1
        rig = MixerRig(spec(H, dim, vdim, window, True), w1, dtype, reader=spec(H2, dim2, vdim2, window2, False), reader_weights=w2)
        for cuts in CUTS + [[at or 60, 1, 1] + [1] * 80 + [330 - 82 - (at or 60)]]:
            got1, got2 = rig.run(h, cuts)
            held(got1, want1, dtype, (at, cuts[:3], "owner"))
            held(got2, want2, dtype, (at, cuts[:3], "reader"))


# ============================================================================ the engine
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("fotulix")
    out = {}
    for n in NAMES:
        folder = make_sharp_model(str(root / n), n, seed=57 + ord(n))
        out[n] = (folder, Plain(folder))
    return out


def close(got, ref, dtype):
    """Whether engine values match the plain model's: every row, in both precisions."""
    return rel_err(got, ref) <= TOL[dtype]


def agrees(got, whole):
    """Whether the bfloat16 engine under some cut gives what it gives for the whole prompt in one step: nine rows of
    ten to a hundredth, the median row to three thousandths (other kernels serve single tokens and prompt portions; their
    sums differ in the last bits, which now and then moves a rounding)."""
    got, whole = got.double().cpu(), whole.double().cpu()
    rows = (got - whole).abs().amax(dim=1) / whole.abs().max()
    return float((rows <= 1e-2).double().mean()) >= 0.9 and float(rows.median()) <= 3e-3


def runner(folder, dtype, max_tokens=512, page=16, seqs=4, pages=None, capture=None):
    from rustinfer_b200.engine.runner import ModelRunner
    return ModelRunner(folder, dtype=dtype, max_model_len=max_tokens, page_size=page,
                       num_pages=pages if pages is not None else max_tokens // page,
                       max_batch_seqs=seqs, max_batch_tokens=max_tokens, capture_sizes=capture)


def run_cuts(r, rid, ids, cuts):
    from rustinfer_b200.engine.runner import StepEntry
    r.open(rid)
    outs, at = [], 0
    for c in cuts:
        outs.append(r.step([StepEntry(rid, ids[at: at + c], list(range(c)))]))
        at += c
    assert at == len(ids)
    r.close(rid)
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_layers_one_by_one(models, name, dtype):
    """The stream after every layer against the plain model's, for a whole prompt and for the same prompt cut in two with
    three single tokens at its end."""
    from rustinfer_b200.engine.runner import StepEntry
    from rustinfer_b200.parts.block import settled_stream
    folder, plain = models[name]
    ids = random_ids(50, CONFIGS[name]["vocab"], 7)
    want = []
    P.forward(plain.cfg, plain.w, ids, want)
    r = runner(folder, dtype)
    taps = []
    r.model.layer_tap = lambda i, hidden: taps.append((i, settled_stream(hidden).cpu()))
    r.open("a")
    r.step([StepEntry("a", ids, [0])])
    r.close("a")
    assert [i for i, _ in taps] == list(range(len(want)))
    for (i, g), w in zip(taps, want):
        assert close(g, w, dtype), i
    taps.clear()
    r.open("b")
    for a, b in ((0, 21), (21, 47), (47, 48), (48, 49), (49, 50)):
        r.step([StepEntry("b", ids[a:b], [0])])
    L = len(want)
    for i, w in enumerate(want):
        got = torch.cat([taps[s * L + i][1] for s in range(5)])
        assert close(got, w, dtype), i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_tail_and_portions(models, name, dtype):
    folder, plain = models[name]
    V = CONFIGS[name]["vocab"]
    r = runner(folder, dtype, page=8 if name == "B" else 16)
    for n, seed in [(130, 1), (61, 2), (1, 3), (3, 4)]:
        ids = random_ids(n, V, seed)
        ref = plain.logits(ids)
        whole = run_cuts(r, "w", ids, [n])
        assert close(whole, ref, dtype)                                        # the first tokens included
        # 32-bit: every cut against the plain model; bfloat16: against the engine's own whole prompt
        same = (lambda got, rows: close(got, ref[:rows], dtype)) if dtype == "float32" else (lambda got, rows: agrees(got, whole[:rows]))
        if n < 40:
            continue
        tail = run_cuts(r, "t", ids, [n - 45] + [1] * 45)                      # windows pass over decoded tokens
        assert same(tail, n)
        cuts, left, sizes = [], n, [2, 7, 1, 16, 2, 33, 24, 5, 2, 64]
        while left:
            c = min(sizes[len(cuts) % len(sizes)], left)
            cuts.append(c)
            left -= c
        assert same(run_cuts(r, "p", ids, cuts), n)
        assert same(run_cuts(r, "two", ids[:40], [2] * 20), 40)
        assert same(run_cuts(r, "one", ids[:40], [1] * 40), 40)                # token by token from the start
    r.cache.check_invariants()
    torch.cuda.synchronize()
    r.check_kernel_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_reuse_pages_and_slots(models, name, dtype):
    """Three state slots and a pool that holds far less than the requests' sum: requests come and go, portions
    of prompts run beside single tokens, and every request's logits are those it has alone."""
    from rustinfer_b200.engine.runner import StepEntry
    folder, plain = models[name]
    V = CONFIGS[name]["vocab"]
    r = runner(folder, dtype, max_tokens=256, page=16, seqs=3, pages=20)
    lens = {"a": 150, "b": 37, "c": 90, "d": 2, "e": 120, "f": 64}
    ids = {k: random_ids(n, V, 100 + i) for i, (k, n) in enumerate(lens.items())}
    at = {k: 0 for k in ids}
    got = {k: [] for k in ids}
    waiting = list(ids)
    live = []
    portion = {"a": [33, 1, 1, 50, 2], "b": [5, 1, 1], "c": [64, 1, 25], "d": [1], "e": [2, 100, 1], "f": [16, 47, 1]}
    turn = 0
    while waiting or live:
        while waiting and len(live) < 3:
            k = waiting.pop(0)
            r.open(k)
            live.append(k)
        entries = []
        for k in live:
            if (turn + ord(k)) % 4 == 3 and len(live) > 1 and len(entries) + 1 < len(live):
                continue                                         # a request sits a step out now and then
            plan = portion[k]
            n = min(plan[min(len(got[k]), len(plan) - 1)], lens[k] - at[k])
            entries.append(StepEntry(k, ids[k][at[k]: at[k] + n], list(range(n))))
        if not entries:
            turn += 1
            continue
        lg = r.step(entries)
        row = 0
        for e in entries:
            n = len(e.tokens)
            got[e.request_id].append(lg[row: row + n])
            row += n
            at[e.request_id] += n
            if at[e.request_id] == lens[e.request_id]:
                r.close(e.request_id)
                live.remove(e.request_id)
        r.cache.check_invariants()
        turn += 1
    for k in ids:
        if dtype == "float32":
            assert close(torch.cat(got[k]), plain.logits(ids[k]), dtype), k
        else:                                                    # against the request alone, whole, on the same engine
            alone = run_cuts(r, "alone-" + k, ids[k], [lens[k]])
            assert agrees(torch.cat(got[k]), alone), k
            if lens[k] >= 30:
                assert close(alone, plain.logits(ids[k]), dtype), k
    torch.cuda.synchronize()
    r.check_kernel_errors()


def test_fp32_logits_do_not_depend_on_the_cut(models):
    """Attention, norms and products add in an order that the cut does not change (the latent layers' batched products may add
    in another one for another count of rows), so the logits agree to rounding."""
    folder, _ = models["A"]
    r = runner(folder, "float32")
    ids = random_ids(90, CONFIGS["A"]["vocab"], 9)
    whole = run_cuts(r, "w", ids, [90])
    assert rel_err(run_cuts(r, "p", ids, [31, 2, 1, 24, 32]), whole) <= 5e-6
    assert rel_err(run_cuts(r, "t", ids, [60] + [1] * 30), whole) <= 5e-6


@pytest.mark.parametrize("name", NAMES)
def test_long_decoding_and_graphs(models, name):
    """300 single tokens after a short prompt, eager and from captured steps: windows pass, their pages are given back, the
    previous token carries, and the logits stay those of the plain model."""
    from rustinfer_b200.engine.runner import StepEntry
    folder, plain = models[name]
    ids = random_ids(310, CONFIGS[name]["vocab"], 5)
    ref = plain.logits(ids)
    for dtype, capture in (("float32", None), ("float32", [1, 2]), ("bfloat16", [1, 2])):
        r = runner(folder, dtype, max_tokens=320, page=16, seqs=2, pages=20, capture=capture)
        r.open("a")
        out = [r.step([StepEntry("a", ids[:10], list(range(10)))])]
        for t in range(10, 310):
            out.append(r.step([StepEntry("a", ids[t: t + 1], [0])]))
        assert close(torch.cat(out), ref, dtype)
        if capture:
            assert r.graph_replays == 300
        r.close("a")
        r.cache.check_invariants()


@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_engine(models, name):
    """`Engine.generate`: scheduler, chunked prefill, continuous batching, device argmax, decode graphs."""
    from rustinfer_b200.engine.engine import Engine
    from rustinfer_b200.sampling.params import SamplingParams
    folder, plain = models[name]
    V = CONFIGS[name]["vocab"]
    prompts = [random_ids(n, V, 50 + n) for n in (45, 3, 70, 1, 26)]
    want = [plain.greedy(p, 12) for p in prompts]
    eng = Engine(folder, dtype="float32", max_batch_seqs=3, max_model_len=128, paged_block_size=16,
                 num_blocks=24, max_batch_tokens=64, chunked_prefill_size=32)
    got = [res.tokens for res in eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))]
    assert got == want
    eng16 = Engine(folder, dtype="bfloat16", max_batch_seqs=3, max_model_len=128, paged_block_size=16,
                   num_blocks=24, max_batch_tokens=64, chunked_prefill_size=32)
    got16 = [res.tokens for res in eng16.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))]
    same = sum(a == b for g, w in zip(got16, want) for a, b in zip(g, w))
    assert same >= 0.5 * 12 * len(prompts), (got16, want)


def test_trace_replay_command(models, tmp_path):
    folder, plain = models["B"]
    V = CONFIGS["B"]["vocab"]
    a, b = random_ids(70, V, 1), random_ids(20, V, 2)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [0, 32]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[33:69], "want": []}, {"id": "b", "tokens": b[:19], "want": [18]}], "end": []},
        {"step": 2, "entries": [{"id": "b", "tokens": b[19:], "want": [0]}, {"id": "a", "tokens": a[69:], "want": [0]}], "end": ["a", "b"]},
    ]
    import numpy as np
    ra, rb = plain.logits(a), plain.logits(b)
    for dtype in DTYPES:
        out = tmp_path / dtype
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=900)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        g0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4")).view(2, V)
        assert rel_err(g0, ra[[0, 32]]) <= TOL[dtype]
        g1 = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4")).view(1, V)
        assert rel_err(g1, rb[[18]]) <= TOL[dtype]
        g2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4")).view(2, V)
        assert rel_err(g2, torch.stack([rb[19], ra[69]])) <= TOL[dtype]


def test_command_line_and_sampler_serve_a_fotulix_folder(models, tmp_path):
    """`bin/rustinfer --config run.toml` on a Fotulix folder: greedy tokens are the plain model's.  Through `Engine`
    with temperature, top-k and top-p: a seeded request gives the same tokens twice, and every drawn token is among
    the most likely at its place."""
    import sys
    from rustinfer_b200.engine.engine import Engine
    from rustinfer_b200.sampling.params import SamplingParams
    folder, plain = models["C"]
    V = CONFIGS["C"]["vocab"]
    prompt = random_ids(21, V, 8)
    (tmp_path / "run.toml").write_text(f"""
model = "{folder}"
dtype = "float32"
max_batch_tokens = 64
max_batch_seqs = 3
max_model_len = 96
paged_block_size = 16
chunked_prefill_size = 8
num_blocks = 18
ignore_eos = true
capture_sizes = [1, 2, 4]

[sampling]
temperature = 0.0
max_tokens = 7

[[request]]
prompt_ids = {prompt}

[[request]]
prompt_ids = {prompt[:5]}
""")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "rustinfer"), "--config", str(tmp_path / "run.toml")],
                       capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-3000:]
    lines = [json.loads(l) for l in p.stdout.splitlines() if l.strip()]
    assert [l["request"] for l in lines] == [0, 1]
    assert lines[0]["tokens"] == plain.greedy(prompt, 7) and lines[1]["tokens"] == plain.greedy(prompt[:5], 7)
    eng = Engine(folder, dtype="float32", max_batch_seqs=3, max_model_len=96, paged_block_size=16, num_blocks=18,
                 max_batch_tokens=64, chunked_prefill_size=8)
    sp = SamplingParams(temperature=0.9, top_k=12, top_p=0.8, seed=11, max_tokens=7, ignore_eos=True)
    first = [r.tokens for r in eng.generate([prompt[:5], prompt], sp)]
    again = [r.tokens for r in eng.generate([prompt[:5], prompt], sp)]
    assert first == again and all(len(t) == 7 for t in first)
    ids = list(prompt[:5])
    for tok in first[0]:
        assert tok in torch.topk(plain.logits(ids)[-1], 12).indices.tolist()
        ids.append(tok)
