"""A plain statement of the Dozotar decoder in float64, one function per mechanism, written from the
design's equations and sharing no code with the package.  Everything runs on whole sequences on the
CPU; nothing is cached, so whatever the engine does with pages, slots and portions is held against
a computation that has none of them.

Notation: h [T, width] is a sublayer's input, p the position of a token (from 0), W x a projection
with W stored [out, in]; a model is (cfg, tensors): config.json's dict and name -> tensor.
"""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def causal_conv(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [T, C], w [C, taps]: y_t = sum_j w[:, j] x_(t - taps + 1 + j) (+ bias), zeros before the start; the
    last column of w meets the current token."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * x[: T - back]
    return y if bias is None else y + bias


def rotate_half(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, H, d]: channel i turns with channel i + dims/2 (i < dims/2) by the angle p * base^(-2i/dims);
    channels from dims on pass."""
    half = dims // 2
    out = x.clone()
    if not half:
        return out
    freq = base ** (-2.0 * torch.arange(half, dtype=F64) / dims)
    ang = (positions.to(F64)[:, None] * freq[None, :])[:, None, :]
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


# ------------------------------------------------------------------------------- attention
def distance_bucket(n: int, rows: int, far: float) -> int:
    """The row of the bias table for a key n positions back: one row a distance for the first half of the rows,
    then logarithmically wider buckets that reach the last row at the distance `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def chunk_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] True where query i sees key j: j <= i, both in one chunk of `size` positions counted from 0."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok & (i // size == j // size) if size else ok


def biased_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: Optional[int],
                     table: torch.Tensor, far: float) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, vd], table [B, H]: score(i, j) = q_i . k_j * scale + table[bucket(i - j)]
    over the keys of the query's chunk, softmax; [T, H, vd]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    qh = q.permute(1, 0, 2)
    kh = k.permute(1, 0, 2).repeat_interleave(H // G, dim=0)
    vh = v.permute(1, 0, 2).repeat_interleave(H // G, dim=0)
    row = torch.tensor([distance_bucket(n, table.shape[0], far) for n in range(T)])
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    s = (qh @ kh.transpose(1, 2)) * scale + table[row[dist]].permute(2, 0, 1)
    s = s.masked_fill(~chunk_mask(T, size)[None], -math.inf)
    return (torch.softmax(s, dim=-1) @ vh).permute(1, 0, 2)


def attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping, eps: float) -> torch.Tensor:
    T, H = h.shape[0], m["heads"]
    G, d = m.get("kv_heads", H), m["dim"]
    vd = m.get("vdim", d)
    q, k, v = (causal_conv(h @ w[x].T, w[x + ".conv"]) for x in ("q", "k", "v"))
    q = (rms(q, eps) * w["q.norm"]).reshape(T, H, d)               # one root mean square for all heads
    k = (rms(k, eps) * w["k.norm"]).reshape(T, G, d)
    size = m["mask"]["size"] if m.get("mask") else None
    o = biased_attention(q, k, v.reshape(T, G, vd), m["scale"], size, w["rel"], m["bias_max"])
    return o.reshape(T, H * vd) @ w["o"].T


# ------------------------------------------------------------------------------- recurrences
def state_walk(key: torch.Tensor, value: torch.Tensor, query: torch.Tensor, decay: torch.Tensor) -> torch.Tensor:
    """key, query [T, H, d], value [T, H, vd], decay [T, H]: S_t = decay_t S_(t-1) + key_t value_t^T per head from
    S = 0; o_t = S_t^T query_t, [T, H, vd]."""
    T, H, d = key.shape
    S = torch.zeros(H, d, value.shape[2], dtype=F64)
    out = []
    for t in range(T):
        S = decay[t][:, None, None] * S + key[t][:, :, None] * value[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, query[t]))
    return torch.stack(out)


def retention(h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping, eps: float) -> torch.Tensor:
    T, H, d = h.shape[0], m["heads"], m["dim"]
    vd = m.get("vdim", d)
    pos = torch.arange(T)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = rotate_half((h @ w["q"].T).reshape(T, H, d), pos, rot["dims"], rot["base"])
    k = rotate_half((h @ w["k"].T).reshape(T, H, d), pos, rot["dims"], rot["base"]) * d ** -0.5
    v = (h @ w["v"].T).reshape(T, H, vd)
    decay = torch.tensor(m["decay"], dtype=F64)[None, :].expand(T, H)
    o = rms(state_walk(k, v, q, decay), eps).reshape(T, H * vd)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """(y * silu(z)) RMS-normed in `parts` equal parts of the last axis, times the weight."""
    g = y * silu(z)
    return rms(g.reshape(*g.shape[:-1], parts, -1), eps).reshape(g.shape) * weight


def mamba2(h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping, eps: float) -> torch.Tensor:
    T, H, vd, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = torch.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, G * N, G * N], dim=-1)
    dt = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=1e9)
    x = x.reshape(T, H, vd)
    B = B.reshape(T, G, N).repeat_interleave(H // G, dim=1)
    C = C.reshape(T, G, N).repeat_interleave(H // G, dim=1)
    y = state_walk(B, dt[:, :, None] * x, C, torch.exp(-torch.exp(w["A_log"]) * dt)) + w["D"][:, None] * x
    return gated_group_norm(y.reshape(T, inner), z, w["norm"], m["norm_groups"], eps) @ w["o"].T


MIXERS = {"attention": attention, "retention": retention, "mamba2": mamba2}


# ------------------------------------------------------------------------------ feed-forward
def gated_ff(h: torch.Tensor, w: Mapping[str, torch.Tensor], act) -> torch.Tensor:
    return (act(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(z: torch.Tensor, top: int, groups: Optional[Mapping] = None):
    """Router logits z [T, E] -> (ids [T, top], weights [T, top]): scores are the softmax over all experts; with
    groups only experts of the `keep` groups with the largest single scores can be chosen; the `top` largest (the
    lower index among equals), weights their scores divided by the scores' sum + 1e-20."""
    s = torch.softmax(z, dim=-1)
    c = s.clone()
    if groups:
        per = z.shape[-1] // groups["count"]
        best = s.reshape(-1, groups["count"], per).max(dim=-1).values
        kept = torch.sort(best, dim=-1, descending=True, stable=True).indices[:, : groups["keep"]]
        allowed = torch.zeros_like(best, dtype=torch.bool).scatter_(1, kept, True).repeat_interleave(per, dim=1)
        c = c.masked_fill(~allowed, -1.0)
    ids = torch.sort(c, dim=-1, descending=True, stable=True).indices[:, :top]
    picked = torch.gather(s, 1, ids)
    return ids, picked / (picked.sum(dim=-1, keepdim=True) + 1e-20)


def sub(tensors: Mapping[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def mixture(h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping) -> torch.Tensor:
    r = m["router"]
    ids, weights = route(h @ w["router"].T, r["top"], r.get("groups"))
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        hit = ids == e
        rows = hit.any(dim=1).nonzero()[:, 0]
        if rows.numel():
            p = (weights * hit).sum(dim=1)[rows]
            out[rows] += p[:, None] * gated_ff(h[rows], sub(w, f"e{e}."), silu)
    if m.get("shared"):
        s = sub(w, "shared.")
        out = out + torch.sigmoid(h @ s["sg"].T) * gated_ff(h, s, silu)
    return out


# ------------------------------------------------------------------------------------- model
def layer(cfg: Mapping, tensors: Mapping[str, torch.Tensor], i: int, x: torch.Tensor) -> torch.Tensor:
    """x <- x + norm1(mixer(x)); x <- x + norm2(ff(x)): the sublayers read x itself, the norms' weight is one number."""
    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]
    w = sub(tensors, f"l{i}.")
    x = x + rms(MIXERS[spec["type"]](x, sub(w, "mix."), spec["mixer"], eps), eps) * w["norm1"]
    mlp = spec.get("mlp")
    if mlp is not None:
        f = sub(w, "mlp.")
        y = gated_ff(x, f, gelu_tanh) if mlp["kind"] == "dense" else mixture(x, f, mlp)
        x = x + rms(y, eps) * w["norm2"]
    return x


def forward(cfg: Mapping, tensors: Mapping[str, torch.Tensor], tokens: List[int], taps: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  `taps`, if a list, receives the stream after every layer."""
    x = tensors["embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)]
    for i in range(len(cfg["layers"])):
        x = layer(cfg, tensors, i, x)
        if taps is not None:
            taps.append(x)
    return (rms(x, cfg["norm"]["eps"]) * tensors["final.norm"].to(F64)) @ tensors["head"].to(F64).T


def greedy(cfg: Mapping, tensors: Mapping[str, torch.Tensor], prompt: List[int], n: int) -> List[int]:
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(torch.argmax(forward(cfg, tensors, seq)[-1]))
        out.append(tok)
        seq.append(tok)
    return out


def read_model_folder(folder: str):
    """(config.json as a dict, tensors by name) of a model folder."""
    import json
    import os
    from safetensors.torch import load_file
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, load_file(os.path.join(folder, "model.safetensors"))
