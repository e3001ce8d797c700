"""A plain statement of the Fotulix decoder in float64, one function per mechanism, written from the
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


# -------------------------------------------------------------------------------- embedding
def bigram_rows(tokens: List[int], mul_prev: int, mul_cur: int, buckets: int) -> List[int]:
    """The row of the bigram table for every token: the last one (`buckets`) for a sequence's first token."""
    return [buckets if t == 0 else (tokens[t - 1] * mul_prev + tokens[t] * mul_cur) % buckets for t in range(len(tokens))]


def embedding(cfg: Mapping, tensors: Mapping[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    emb = cfg.get("embedding") or {}
    x = tensors["embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)] * emb.get("scale", 1.0)
    b = emb.get("bigram")
    if b:
        rows = bigram_rows(tokens, b["mul_prev"], b["mul_cur"], b["buckets"])
        x = x + tensors["bigram"].to(F64)[torch.tensor(rows, dtype=torch.long)]
    return x


# -------------------------------------------------------------------------------- positions
def frequencies(rot: Mapping) -> List[float]:
    return [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]


def banded_frequencies(rot: Mapping) -> List[float]:
    """Wavelengths below original/high keep their frequency, those above original/low have it divided by factor, the
    band between blends the two linearly in original/wavelength."""
    s = rot.get("scaling")
    out = []
    for f in frequencies(rot):
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - t) * f / s["factor"] + t * f
        out.append(f)
    return out


def yarn_frequencies(rot: Mapping):
    """(frequencies, factor on cos and sin): pair i keeps its frequency below the pair that turns `fast` times over the
    original length, has it divided by factor above the pair that turns `slow` times, and a linear ramp between."""
    s, dims = rot.get("scaling"), rot["dims"]
    freq = frequencies(rot)
    if not s:
        return freq, 1.0

    def pair_of(turns: float) -> float:
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))
    lo = max(math.floor(pair_of(s["fast"])), 0)
    hi = min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x: torch.Tensor, freq: List[float], magnitude: float = 1.0) -> torch.Tensor:
    """x [T, ..., d], token t at position t: channels (2i, 2i+1) turn by t * freq_i, cos and sin times `magnitude`; the
    channels behind the pairs pass."""
    dims = 2 * len(freq)
    if not dims:
        return x
    out = x.clone()
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor(freq, dtype=F64)[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    c, s = (torch.cos(ang) * magnitude).reshape(shape), (torch.sin(ang) * magnitude).reshape(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def query_temperature(T: int, coef: float, every: float) -> torch.Tensor:
    """[T]: 1 + coef ln(floor((p + 1) / every) + 1) at position p."""
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in range(T)], dtype=F64)


def distance_bucket(n: int, rows: int, far: float) -> int:
    """The row of the bias table for a key n positions back: one row a distance for the first half of the rows,
    then logarithmically wider buckets that reach the last row at the distance `far`."""
    half = rows / 2
    if n < half:
        return n
    return min(rows - 1, int(half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


# -------------------------------------------------------------------------------- attention
def visible(T: int, window: Optional[int]) -> torch.Tensor:
    """[T, T] True where query i sees key j: 0 <= i - j (< window where there is one)."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < window) if window else back >= 0


def softmax_with_sink(scores: torch.Tensor, mask: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """Softmax over the visible keys of scores [H, T, T]; with `sink` [H] the denominator also holds
    exp(sink_h), a term without key or value."""
    s = scores.masked_fill(~mask[None], -math.inf)
    m = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink.reshape(-1, 1, 1))
    e = torch.exp(s - m)
    den = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink.reshape(-1, 1, 1) - m)
    return e / den


def grouped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, bias: Optional[torch.Tensor] = None,
                      sink: Optional[torch.Tensor] = None, window: Optional[int] = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, vd]: query head h reads head h // (H/G); score = q.k * scale + bias [H, T, T];
    [T, H, vd]."""
    H, G = q.shape[1], k.shape[1]
    kh = k.permute(1, 0, 2).repeat_interleave(H // G, dim=0)
    vh = v.permute(1, 0, 2).repeat_interleave(H // G, dim=0)
    s = (q.permute(1, 0, 2) @ kh.transpose(1, 2)) * scale
    if bias is not None:
        s = s + bias
    return (softmax_with_sink(s, visible(q.shape[0], window), sink) @ vh).permute(1, 0, 2)


def bias_by_distance(table: torch.Tensor, far: float, T: int) -> torch.Tensor:
    """table [rows, H] -> [H, T, T], entry (i, j) the bias of a key i - j positions back (of 0 for later keys)."""
    row = torch.tensor([distance_bucket(n, table.shape[0], far) for n in range(T)])
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    return table[row[back]].permute(2, 0, 1)


def gate_heads(o: torch.Tensor, h: torch.Tensor, g: torch.Tensor) -> torch.Tensor:
    """o [T, H, vd]: head h's output times sigmoid of the h-th of H numbers W_g h; flat [T, H*vd]."""
    return (o * torch.sigmoid(h @ g.T)[:, :, None]).reshape(o.shape[0], -1)


def attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping) -> torch.Tensor:
    """No rotation: a query temperature by position and a learned bias by the distance's bucket; biased projections."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    G, vd = m.get("kv_heads", H), m.get("vdim", d)
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, d)
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, d)
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, vd)
    if m.get("q_temp"):
        q = q * query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    o = grouped_attention(q, k, v, m["scale"], bias=bias_by_distance(w["rel"], m["bias_max"], T))
    return gate_heads(o, h, w["g"]) @ w["o"].T


def attention_2(h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping) -> torch.Tensor:
    """Rotated queries and keys, a learned sink a head."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    G, vd = m.get("kv_heads", H), m.get("vdim", d)
    freq = banded_frequencies(m["rot"]) if m.get("rot") else []
    q = rotate_pairs((h @ w["q"].T).reshape(T, H, d), freq)
    k = rotate_pairs((h @ w["k"].T).reshape(T, G, d), freq)
    o = grouped_attention(q, k, (h @ w["v"].T).reshape(T, G, vd), m["scale"], sink=w["sink"])
    return gate_heads(o, h, w["g"]) @ w["o"].T


def latent_rows(h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping, eps: float):
    """(c [T, rank], rotated key part [T, rot_dim]): what a latent layer caches of its input."""
    rank = m["kv_rank"]
    freq, mag = yarn_frequencies(m["rot"])
    low = h @ w["dkv"].T
    return rms(low[:, :rank], eps) * w["dkv.norm"], rotate_pairs(low[:, rank:], freq, mag)


def latent_attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping, eps: float, rows=None) -> torch.Tensor:
    """`rows`: another latent layer's (c, rotated key part), in place of this layer's own."""
    T, H, d, rd, vd = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = latent_rows(h, w, m, eps) if rows is None else rows
    freq, mag = yarn_frequencies(m["rot"])
    q = (h @ w["q"].T).reshape(T, H, d + rd)
    q_plain, q_rot = q[..., :d], rotate_pairs(q[..., d:], freq, mag)
    k_plain = (c @ w["uk"].T).reshape(T, H, d)
    v = (c @ w["uv"].T).reshape(T, H, vd)
    s = torch.einsum("thd,shd->hts", q_plain, k_plain) + torch.einsum("thr,sr->hts", q_rot, k_rot)
    window = m["mask"]["size"] if m.get("mask") else None
    p = softmax_with_sink(s * m["scale"], visible(T, window), None)
    return gate_heads(torch.einsum("hts,shv->thv", p, v), h, w["g"]) @ w["o"].T


# ------------------------------------------------------------------------------ the rest of a layer
def gated_ff(h: torch.Tensor, w: Mapping[str, torch.Tensor]) -> torch.Tensor:
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def token_side(x: torch.Tensor, e: torch.Tensor, w: Mapping[str, torch.Tensor], eps: float) -> torch.Tensor:
    """x [T, width] the stream, e [T, dim] the tokens' rows of this layer: rms(proj(gelu_tanh(gate x) * e)) * norm."""
    return rms((gelu_tanh(x @ w["gate"].T) * e) @ w["proj"].T, eps) * w["norm"]


def sub(tensors: Mapping[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def layer(cfg: Mapping, tensors: Mapping[str, torch.Tensor], i: int, x: torch.Tensor, tokens: List[int], latents: dict) -> torch.Tensor:
    """`latents`: layer number -> what that latent layer caches of this sequence (filled here)."""
    spec, eps, m = cfg["layers"][i], cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    w = sub(tensors, f"l{i}.")
    mix, mw = spec["mixer"], sub(w, "mix.")
    h = rms(x, eps) * (1.0 + w["norm1"])
    if spec["type"] == "attention":
        y = attention(h, mw, mix)
    elif spec["type"] == "attention_2":
        y = attention_2(h, mw, mix)
    elif mix.get("kv_from") is not None:
        y = latent_attention(h, mw, mix, eps, latents[mix["kv_from"]])
    else:
        latents[i] = latent_rows(h, mw, mix, eps)
        y = latent_attention(h, mw, mix, eps)
    x = x + m * rms(y, eps) * (1.0 + w["norm1b"])
    if spec.get("mlp") is not None:
        y = gated_ff(rms(x, eps) * (1.0 + w["norm2"]), sub(w, "mlp."))
        x = x + m * rms(y, eps) * (1.0 + w["norm2b"])
    side = cfg.get("token_side")
    if side:
        dim = side["dim"]
        e = tensors["side.embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)][:, i * dim: (i + 1) * dim]
        x = x + m * token_side(x, e, sub(w, "side."), eps)
    return x


def forward(cfg: Mapping, tensors: Mapping[str, torch.Tensor], tokens: List[int], taps: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  `taps`, if a list, receives the stream after every layer."""
    x = embedding(cfg, tensors, tokens)
    latents: dict = {}
    for i in range(len(cfg["layers"])):
        x = layer(cfg, tensors, i, x, tokens, latents)
        if taps is not None:
            taps.append(x)
    return (rms(x, cfg["norm"]["eps"]) * (1.0 + tensors["final.norm"].to(F64))) @ tensors["head"].to(F64).T


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
