"""Shared by the Dozotar tests: small configurations that differ from one another in every size, constant
and layer order, weights that make faults show, model folders, the plain model's logits."""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Sequence

import torch

import plain_dozotar


def _attention(heads, kv, dim, vdim, conv, scale, far, mask):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "bias_max": far}
    if mask:
        m["mask"] = {"size": mask}
    return {"type": "attention", "mixer": m}


def _retention(heads, dim, vdim, decay, rot=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "retention", "mixer": m}


def _mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def _moe(ff, experts, top, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        m["shared"] = {"ff": shared}
    return m


# A: attention first, values wider than keys, chunks of 20 positions (a page and a quarter), three taps, a table of 8 rows;
#    a state-space layer with three groups and four norm parts and two taps; retention rotated on 8 of its 20 channels, no
#    feed-forward
# B: a state-space layer of one group normed as a whole; experts without groups and without a shared one; chunks equal to
#    the page; one expert of three beside a shared one; as many kv heads as heads
# C: one retention head, rotated whole; attention without chunks over one kv head, keys wider than values, one tap (no
#    state), a table of 5 rows; every expert used by every token; a state-space layer with a group a head, sizes that are
#    no multiple of anything, one tap, a norm part a head
# D: every attention size a multiple of 16, so that the bfloat16 engine's prompt portions run on the tensor-core attention;
#    eight heads on one kv head, whose single tokens run there too; chunks of 50 (three pages and two tokens); retention
#    without rotation; all groups kept
# E: a width and feed-forwards that are no multiple of eight (nothing runs on the tensor cores but what pads), odd sizes
#    everywhere, a table that ends at 9 positions back, a state-space mixer whose step sizes start at an odd column
# F: no attention at all: every cache is a state
CONFIGS = {
    "A": {"architecture": "Dozotar", "width": 96, "vocab": 211, "norm": {"eps": 1e-5}, "layers": [
        dict(_attention(4, 2, 24, 40, 3, 0.3, 50.0, 20), mlp={"kind": "dense", "ff": 136}),
        dict(_mamba(6, 20, 24, 3, 2, 4), mlp=_moe(40, 8, 3, (4, 2), 56)),
        dict(_retention(3, 20, 12, [0.99, 0.9, 0.5], (8, 500.0)), mlp=None)]},
    "B": {"architecture": "Dozotar", "width": 128, "vocab": 300, "norm": {"eps": 1e-6}, "layers": [
        dict(_mamba(4, 32, 16, 1, 4, 1), mlp=_moe(64, 5, 2)),
        dict(_attention(2, 2, 32, 32, 4, 0.2, 100.0, 16), mlp=_moe(72, 3, 1, None, 24))]},
    "C": {"architecture": "Dozotar", "width": 64, "vocab": 97, "norm": {"eps": 3e-6}, "layers": [
        dict(_retention(1, 40, 24, [0.97], (40, 10000.0)), mlp={"kind": "dense", "ff": 40}),
        dict(_attention(6, 1, 24, 8, 1, 0.4, 30.0, None), mlp=_moe(24, 3, 3, None, 32)),
        dict(_mamba(5, 7, 9, 5, 1, 5), mlp=None)]},
    "D": {"architecture": "Dozotar", "width": 80, "vocab": 150, "norm": {"eps": 2e-5}, "layers": [
        dict(_attention(4, 2, 16, 32, 2, 0.25, 200.0, 50), mlp=_moe(48, 6, 2, (2, 2), 16)),
        dict(_retention(2, 64, 48, [0.999, 0.95]), mlp=_moe(32, 8, 2, (4, 1))),
        dict(_attention(8, 1, 32, 16, 3, 0.3, 64.0, 37), mlp={"kind": "dense", "ff": 64}),
        dict(_mamba(4, 16, 64, 2, 4, 2), mlp=_moe(40, 6, 2, (3, 2), 48))]},
    "E": {"architecture": "Dozotar", "width": 92, "vocab": 101, "norm": {"eps": 1e-4}, "layers": [
        dict(_attention(3, 3, 23, 9, 4, 0.3, 9.0, 21), mlp=_moe(22, 7, 4, None, 13)),
        dict(_mamba(3, 6, 15, 1, 3, 3), mlp={"kind": "dense", "ff": 30}),
        dict(_attention(5, 1, 40, 24, 2, 0.2, 77.0, 64), mlp=_moe(26, 6, 1, (6, 1), None)),
        dict(_retention(3, 14, 10, [0.98, 0.7, 0.999], (6, 50.0)), mlp=_moe(18, 4, 2, (2, 1), 20))]},
    "F": {"architecture": "Dozotar", "width": 48, "vocab": 80, "norm": {"eps": 1e-5}, "layers": [
        dict(_mamba(2, 24, 16, 2, 4, 1), mlp=None),
        dict(_retention(2, 16, 16, [0.95, 0.99], (16, 1000.0)), mlp=_moe(16, 4, 2)),
        dict(_mamba(3, 16, 20, 1, 2, 3), mlp={"kind": "dense", "ff": 64})]},
}
REL_ROWS = {("A", 0): 8, ("B", 1): 16, ("C", 1): 5, ("D", 0): 32, ("D", 2): 12, ("E", 0): 6, ("E", 2): 16}


def tensor_shapes(name: str) -> Dict[str, tuple]:
    """Names and shapes of a checkpoint, written out here so that the tests do not lean on the framework's own list."""
    cfg = CONFIGS[name]
    d, v = cfg["width"], cfg["vocab"]
    s = {"embed": (v, d), "head": (v, d), "final.norm": ()}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        s[p + "norm1"] = ()
        H = m["heads"]
        if layer["type"] == "attention":
            G, dim, vd, taps = m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            s.update({x + "q": (H * dim, d), x + "k": (G * dim, d), x + "v": (G * vd, d), x + "q.norm": (H * dim,),
                      x + "k.norm": (G * dim,), x + "q.conv": (H * dim, taps), x + "k.conv": (G * dim, taps),
                      x + "v.conv": (G * vd, taps), x + "rel": (REL_ROWS[(name, i)], H), x + "o": (d, H * vd)})
        elif layer["type"] == "retention":
            s.update({x + "q": (H * m["dim"], d), x + "k": (H * m["dim"], d), x + "v": (H * m["vdim"], d),
                      x + "g": (H * m["vdim"], d), x + "o": (d, H * m["vdim"])})
        else:
            inner = H * m["vdim"]
            C = inner + 2 * m["groups"] * m["state"]
            s.update({x + "in": (inner + C + H, d), x + "conv": (C, m["conv"]), x + "conv.b": (C,), x + "dt_bias": (H,),
                      x + "A_log": (H,), x + "D": (H,), x + "norm": (inner,), x + "o": (d, inner)})
        mlp = layer["mlp"]
        if mlp is None:
            continue
        s[p + "norm2"] = ()
        y = p + "mlp."
        if mlp["kind"] == "dense":
            s.update({y + "gate": (mlp["ff"], d), y + "up": (mlp["ff"], d), y + "down": (d, mlp["ff"])})
            continue
        ff, E = mlp["expert"]["ff"], mlp["router"]["experts"]
        s[y + "router"] = (E, d)
        for e in range(E):
            s.update({y + f"e{e}.gate": (ff, d), y + f"e{e}.up": (ff, d), y + f"e{e}.down": (d, ff)})
        if mlp.get("shared"):
            sf = mlp["shared"]["ff"]
            s.update({y + "shared.gate": (sf, d), y + "shared.up": (sf, d), y + "shared.down": (d, sf), y + "shared.sg": (1, d)})
    return s


def sharp_weights(name: str, seed: int, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Matrices of size 1/sqrt(fan_in) (the router twice that, so that the choice of experts is peaked), norm weights of q
    and k of size 2 (the attention is peaked), bias tables with a spread of 2 (a wrong bucket shows), the layers' one norm
    number spread around 0.8, step sizes and decays from short to long memories."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in tensor_shapes(name).items():
        parts = n.split(".")
        leaf = parts[-1]
        if shape == ():
            t = 0.8 + 0.3 * torch.randn(shape, generator=g)
        elif leaf in ("rel",):
            t = 2.0 * torch.randn(shape, generator=g)
        elif leaf == "conv":
            t = 0.5 * torch.randn(shape, generator=g)
            t[:, -1] += 0.7
        elif leaf == "b":
            t = 0.3 * torch.randn(shape, generator=g)
        elif leaf == "dt_bias":
            t = torch.randn(shape, generator=g) - 2.0
        elif leaf == "A_log":
            t = torch.randn(shape, generator=g)
        elif leaf == "D":
            t = torch.randn(shape, generator=g)
        elif leaf == "norm":
            t = (2.0 if parts[-2] in ("q", "k") else 1.0) + 0.3 * torch.randn(shape, generator=g)
        elif n == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
            if leaf == "router":
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
        self.cfg, self.w = plain_dozotar.read_model_folder(folder)
        self._memo = {}

    def logits(self, ids: Sequence[int]) -> torch.Tensor:
        key = tuple(ids)
        if key not in self._memo:
            self._memo[key] = plain_dozotar.forward(self.cfg, self.w, list(ids))
        return self._memo[key]

    def greedy(self, prompt: Sequence[int], n: int) -> List[int]:
        ids, out = list(prompt), []
        for _ in range(n):
            t = int(torch.argmax(self.logits(ids)[-1]))
            out.append(t)
            ids.append(t)
        return out
