"""Shared by the Fotulix tests: small configurations that differ from one another in every size, constant
and layer order, weights that make faults show, model folders, the plain model's logits."""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Sequence

import torch

import plain_fotulix


def _attention(heads, kv, dim, vdim, scale, far, temp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": far}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m}


def _rotary(heads, kv, dim, vdim, scale, rot=None, bands=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if bands:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    return {"type": "attention_2", "mixer": m}


def _latent(heads, dim, rot_dim, vdim, rank, scale, base, window=None, yarn=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base}}
    if yarn:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def _ff(ff):
    return {"kind": "dense", "ff": ff}


# A: every mixer; values wider than keys; a reader with a wider window than the owner of the rows, more heads and other
#    sizes; a layer without a feed-forward; the temperature steps every 16 positions
# B: a latent layer first, its window as long as a page (8 where the tests say so); two readers, one narrower and one as
#    wide, one of them last; no scaling, no bigrams, no input by token; no temperature
# C: odd sizes everywhere (nothing is a multiple of eight), a table that ends 9 positions back, one head on one, a reader
#    that sees every row of an owner with a window; rotation of the whole head; temperature every 3 positions
# D: every attention size a multiple of 16, so that the bfloat16 engine's prompt portions run on the tensor-core attention;
#    eight heads on one kv head and twelve latent heads, whose single tokens run there too; windows of three pages and two
# E: only latent layers; no `residual_mult`, no `embedding`: scale 1 and no pairs; a temperature nowhere
# F: no rotation in `attention_2`; bigrams with one bucket and with factors that overflow 32 bits; window of one key
CONFIGS = {
    "A": {"architecture": "Fotulix", "width": 96, "vocab": 211, "norm": {"eps": 1e-5}, "residual_mult": 0.7,
          "embedding": {"scale": 3.0, "bigram": {"buckets": 61, "mul_prev": 17, "mul_cur": 5}}, "token_side": {"dim": 12}, "layers": [
        dict(_attention(4, 2, 24, 40, 0.3, 50.0, (0.7, 16)), mlp=_ff(136)),
        dict(_latent(3, 16, 8, 20, 24, 0.25, 3000.0, 20, (3.0, 64, 8.0, 0.5)), mlp=None),
        dict(_rotary(4, 1, 24, 8, 0.25, (8, 500.0), (4.0, 1.0, 4.0, 48)), mlp=_ff(72)),
        dict(_latent(5, 10, 8, 12, 24, 0.3, 3000.0, 37, (3.0, 64, 8.0, 0.5), kv_from=1), mlp=_ff(64)),
        dict(_attention(6, 3, 16, 24, 0.35, 30.0, (0.4, 50)), mlp=_ff(40))]},
    "B": {"architecture": "Fotulix", "width": 128, "vocab": 300, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
          "embedding": {"scale": 2.0}, "layers": [
        dict(_latent(8, 32, 16, 24, 32, 0.2, 10000.0, 16), mlp=_ff(96)),
        dict(_latent(2, 16, 16, 32, 32, 0.3, 10000.0, 9, kv_from=0), mlp=_ff(64)),
        dict(_attention(2, 2, 32, 32, 0.25, 100.0), mlp=_ff(128)),
        dict(_rotary(2, 2, 32, 32, 0.25, (16, 10000.0)), mlp=_ff(72)),
        dict(_latent(9, 8, 16, 16, 32, 0.3, 10000.0, 16, kv_from=0), mlp=None)]},
    "C": {"architecture": "Fotulix", "width": 92, "vocab": 101, "norm": {"eps": 1e-4}, "residual_mult": 0.35,
          "embedding": {"scale": 2.5, "bigram": {"buckets": 7, "mul_prev": 1, "mul_cur": 1}}, "token_side": {"dim": 7}, "layers": [
        dict(_rotary(1, 1, 40, 24, 0.2, (40, 70.0), (2.0, 2.0, 3.0, 20)), mlp=_ff(30)),
        dict(_attention(3, 3, 23, 9, 0.3, 9.0, (1.5, 3)), mlp=_ff(22)),
        dict(_latent(3, 7, 4, 9, 20, 0.4, 40.0, 11, (5.0, 30, 2.0, 1.0)), mlp=_ff(26)),
        dict(_latent(1, 5, 4, 3, 20, 0.5, 40.0, None, (5.0, 30, 2.0, 1.0), kv_from=2), mlp=None)]},
    "D": {"architecture": "Fotulix", "width": 80, "vocab": 150, "norm": {"eps": 2e-5}, "residual_mult": 0.4,
          "embedding": {"scale": 4.0, "bigram": {"buckets": 97, "mul_prev": 31, "mul_cur": 11}}, "token_side": {"dim": 16}, "layers": [
        dict(_attention(8, 1, 16, 32, 0.3, 200.0, (0.2, 64)), mlp=_ff(48)),
        dict(_latent(12, 16, 16, 16, 80, 0.25, 20000.0, 50, (8.0, 100, 16.0, 1.0)), mlp=_ff(64)),
        dict(_rotary(6, 2, 32, 16, 0.3, (24, 9000.0), (4.0, 1.0, 4.0, 64)), mlp=_ff(80)),
        dict(_latent(8, 32, 16, 48, 80, 0.2, 20000.0, 33, (8.0, 100, 16.0, 1.0), kv_from=1), mlp=_ff(64)),
        dict(_rotary(4, 2, 64, 48, 0.2, (64, 100.0)), mlp=_ff(64))]},
    "E": {"architecture": "Fotulix", "width": 64, "vocab": 97, "norm": {"eps": 3e-6}, "token_side": {"dim": 20}, "layers": [
        dict(_latent(1, 24, 4, 16, 20, 0.3, 100.0, 5), mlp=_ff(40)),
        dict(_latent(4, 12, 8, 8, 24, 0.3, 1000.0, 64, (2.0, 512, 32.0, 1.0)), mlp=_ff(24)),
        dict(_latent(2, 24, 4, 16, 20, 0.3, 100.0, 6, kv_from=0), mlp=_ff(40))]},
    "F": {"architecture": "Fotulix", "width": 48, "vocab": 80, "norm": {"eps": 1e-5}, "residual_mult": 0.8,
          "embedding": {"scale": 1.5, "bigram": {"buckets": 1000, "mul_prev": 2147483647, "mul_cur": 1099511627791}}, "layers": [
        dict(_rotary(2, 1, 16, 24, 0.4), mlp=None),
        dict(_latent(2, 16, 8, 16, 24, 0.3, 50.0, 1), mlp=_ff(64)),
        dict(_attention(4, 4, 8, 16, 0.5, 3.0, (0.9, 100)), mlp=_ff(40))]},
}
REL_ROWS = {("A", 0): 8, ("A", 4): 6, ("B", 2): 16, ("C", 1): 6, ("D", 0): 32, ("F", 2): 4}


def tensor_shapes(name: str) -> Dict[str, tuple]:
    """Names and shapes of a checkpoint, written out here so that the tests do not lean on the framework's own list."""
    cfg = CONFIGS[name]
    d, v = cfg["width"], cfg["vocab"]
    s = {"embed": (v, d), "head": (v, d), "final.norm": (d,)}
    bigram = cfg.get("embedding", {}).get("bigram")
    if bigram:
        s["bigram"] = (bigram["buckets"] + 1, d)
    side = cfg.get("token_side", {}).get("dim")
    if side:
        s["side.embed"] = (v, side * len(cfg["layers"]))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        s.update({p + "norm1": (d,), p + "norm1b": (d,)})
        H, dim, vd = m["heads"], m["dim"], m["vdim"]
        s.update({x + "g": (H, d), x + "o": (d, H * vd)})
        if layer["type"] == "latent_attention":
            rank, rd = m["kv_rank"], m["rot_dim"]
            s.update({x + "q": (H * (dim + rd), d), x + "uk": (H * dim, rank), x + "uv": (H * vd, rank)})
            if "kv_from" not in m:
                s.update({x + "dkv": (rank + rd, d), x + "dkv.norm": (rank,)})
        else:
            G = m["kv_heads"]
            s.update({x + "q": (H * dim, d), x + "k": (G * dim, d), x + "v": (G * vd, d)})
            if layer["type"] == "attention":
                s.update({x + "q.b": (H * dim,), x + "k.b": (G * dim,), x + "v.b": (G * vd,), x + "rel": (REL_ROWS[(name, i)], H)})
            else:
                s[x + "sink"] = (H,)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            s.update({p + "norm2": (d,), p + "norm2b": (d,), p + "mlp.gate": (ff, d), p + "mlp.up": (ff, d), p + "mlp.down": (d, ff)})
        if side:
            s.update({p + "side.gate": (side, d), p + "side.proj": (d, side), p + "side.norm": (d,)})
    return s


def sharp_weights(name: str, seed: int, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Matrices of size 1/sqrt(fan_in) (queries, keys and the latent's up-projection of keys twice that, so that the attention
    is peaked), norm weights around zero with a spread of 0.3, bias tables with a spread of 2 (a wrong bucket shows), sinks
    around 1, biases of 0.5, tables of a size that shows in the stream.  (Every sublayer's output is divided by its own root mean
    square: a stream that is large beside what the few-channel sublayers add keeps bfloat16's rounding of small outputs from
    taking over a row.)"""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in tensor_shapes(name).items():
        leaf = n.split(".")[-1]
        if n in ("embed", "bigram", "side.embed"):
            t = torch.randn(shape, generator=g) * (4.0 if n == "embed" and "embedding" not in CONFIGS[name] else 1.0)
        elif n.endswith(("dkv.norm", "side.norm")):
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif leaf in ("norm1", "norm1b", "norm2", "norm2b", "norm"):
            t = 0.3 * torch.randn(shape, generator=g)
        elif leaf == "rel":
            t = 2.0 * torch.randn(shape, generator=g)
        elif leaf == "sink":
            t = 1.0 + torch.randn(shape, generator=g)
        elif leaf == "b":
            t = 0.5 * torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
            if leaf in ("q", "k", "uk"):
                t = t * 2.0
        out[n] = t.to(dtype)
    return out


def write_model(folder: str, name: str, weights: Dict[str, torch.Tensor]) -> str:
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(CONFIGS[name], f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(folder, "model.safetensors"))
    return folder


def make_sharp_model(folder: str, name: str, seed: int = 0) -> str:
    return write_model(folder, name, sharp_weights(name, seed))


class Plain:
    """The plain implementation over one model folder, with per-sequence memo."""

    def __init__(self, folder: str):
        self.cfg, self.w = plain_fotulix.read_model_folder(folder)
        self._memo = {}

    def logits(self, ids: Sequence[int]) -> torch.Tensor:
        key = tuple(ids)
        if key not in self._memo:
            self._memo[key] = plain_fotulix.forward(self.cfg, self.w, list(ids))
        return self._memo[key]

    def greedy(self, prompt: Sequence[int], n: int) -> List[int]:
        ids, out = list(prompt), []
        for _ in range(n):
            t = int(torch.argmax(self.logits(ids)[-1]))
            out.append(t)
            ids.append(t)
        return out


class MixerRig:
    """One mixer part by itself on the GPU: caches of its own, pages scrambled and poisoned, a `StepContext` made by hand for
    every portion.  `reader`: a second part that reads the first one's cache and writes nothing."""

    def __init__(self, spec, weights, dtype, max_len=512, page=8, reader=None, reader_weights=None):
        import rustinfer_b200.models.decoder  # noqa: F401  (registers the built-in parts)
        from rustinfer_b200.parts.base import BuildContext, MIXERS
        self.dev = torch.device("cuda:0")
        self.ctx = BuildContext(self.dev, dtype, max_len, page, max_batch_seqs=4)
        self.page, self.dtype = page, dtype

        def build(s, w):
            part = MIXERS.build(s)
            part.prepare(self.ctx)
            assert set(part.param_decls()) == set(w)
            part.load({k: v.to(dtype).to(self.dev) for k, v in w.items()})
            return part
        self.part = build(spec, weights)
        self.reader = build(reader, reader_weights) if reader is not None else None
        need = self.part.cache_need()
        self.pages = max_len // page
        if need.plain:
            shape = (self.pages + 3, 2, need.num_kv_heads, page, need.head_dim)
        else:
            shape = (self.pages + 3, page * need.elems_per_token())
        self.kv = torch.full(shape, 1e4, dtype=dtype, device=self.dev)
        self.table = torch.randperm(self.pages, generator=torch.Generator().manual_seed(3)) + 2

    def run(self, h: torch.Tensor, cuts: Sequence[int]):
        """h [T, width] of one request in portions; the outputs of the part (and of the reader, if any)."""
        import numpy as np
        from rustinfer_b200.parts.base import GroupStep, PagedLayerCache, StepContext, StepShape
        i32 = lambda x: torch.as_tensor(x, dtype=torch.int32, device=self.dev)
        outs, at = [[], []], 0
        for n in cuts:
            pos = torch.arange(at, at + n)
            shape = StepShape(np.array([n]), np.array([at]), np.array([0, n]), np.array([at + n]), np.array([0]))
            needs = list(self.part.step_indices()) + (list(self.reader.step_indices()) if self.reader is not None else [])
            indices = {need.key: tuple(i32(a) for a in need.build(shape)) for need in needs}
            group = GroupStep(i32(self.table[None].numpy()), i32((self.table[pos // self.page] * self.page + pos % self.page).numpy()))
            step = StepContext(n, 1, i32([0] * n), i32(pos.numpy()), i32([0, n]), i32([at + n]), i32([0]), [group], [], n, at + n,
                               n == 1, indices)
            x = h[at: at + n].to(self.dtype).to(self.dev).contiguous()
            outs[0].append(self.part.forward(x, step, PagedLayerCache(self.kv, 0, True)).double().cpu())
            if self.reader is not None:
                outs[1].append(self.reader.forward(x, step, PagedLayerCache(self.kv, 0, False)).double().cpu())
            at += n
        assert at == h.shape[0]
        whole = [torch.cat(o) for o in outs if o]
        return whole if self.reader is not None else whole[0]
