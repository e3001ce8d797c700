"""A mixer that is a state-space recurrence with step sizes (Dao and Gu, "Transformers are SSMs: Generalized Models and
Efficient Algorithms Through Structured State Space Duality", known as Mamba-2):

    [z | x | B | C | dt] = W_in h                      z, x: H heads of vd channels; B, C: G groups of N; dt: H
    x, B, C <- silu(conv([x | B | C]))                 a short causal convolution a channel, with a bias
    dt <- softplus(dt + dt_bias),  a = exp(-exp(A_log) dt)
    S_t = a_t S_(t-1) + dt_t B_t x_t^T,  y_t = S_t^T C_t + D x_t       head h reads group h // (H / G)
    out = W_o ( rms_part(y * silu(z)) * w )            the gated row normed in equal parts

The state [N, vd] of a head (fp32, zero for a new request) and the convolution's last taps - 1 inputs sit in slots of two
fixed-state cache groups.  The input product leaves fp32; the convolution with its activation, the step sizes, decays, the
recurrence, the gate and the norm are fp32 in both engines, and what W_o reads is rounded once.  The walk is the
one-decay-a-head form of the linear-attention recurrences (keys B, values dt x, queries C).  The reference engine has no
recurrent mixer (crates/infer-worker/src/components/attention.rs is its only one).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..ops import kernels as K
from .base import FixedState, Mixer, ParamDecl, StepContext, register_mixer
from .linear import Linear
from .short_conv import ConvState


@register_mixer("mamba2")
class Mamba2(Mixer):
    """params: hidden_size, num_heads, value_dim, state_dim, groups, conv_taps, norm_groups, norm_eps, tensor_names (local
    name -> name in the file).  Tensors: in [2 H vd + 2 G N + H, hidden] (rows z, x, B, C, dt); conv [H vd + 2 G N, taps],
    conv.b; dt_bias, A_log, D [H]; norm [H vd]; o [hidden, H vd]."""
    graph_safe = True

    def __init__(self, params):
        super().__init__(params)
        p = params
        self.hidden, self.H, self.vd = int(p["hidden_size"]), int(p["num_heads"]), int(p["value_dim"])
        self.N, self.G = int(p["state_dim"]), int(p.get("groups", 1))
        self.norm_groups, self.norm_eps = int(p.get("norm_groups", 1)), float(p["norm_eps"])
        self.tensor_names = dict(p.get("tensor_names") or {})
        self.inner = self.H * self.vd
        self.channels = self.inner + 2 * self.G * self.N
        if self.H % self.G or self.inner % self.norm_groups:
            raise ValueError("groups divide the heads, and norm_groups the channels")
        if not 1 <= self.N <= 512:
            raise ValueError(f"state size {self.N}: the recurrence kernels take key sizes up to 512")
        self.conv = ConvState(self.channels, int(p["conv_taps"]), activation="silu")

    def _name(self, local: str) -> str:
        return self.tensor_names.get(local, local)

    def param_decls(self) -> Dict[str, ParamDecl]:
        n, C = self._name, self.channels
        return {n("in"): ParamDecl((self.inner + C + self.H, self.hidden)),
                n("conv"): ParamDecl((C, self.conv.taps)), n("conv.b"): ParamDecl((C,), init="zeros"),
                n("dt_bias"): ParamDecl((self.H,)), n("A_log"): ParamDecl((self.H,)), n("D"): ParamDecl((self.H,), init="ones"),
                n("norm"): ParamDecl((self.inner,), init="ones"), n("o"): ParamDecl((self.hidden, self.inner))}

    def cache_need(self):
        return (self.conv.need(), FixedState((self.H, self.vd, K.recurrent_state_rows(self.N)), "float32"))

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self._name
        f32 = lambda name: tensors[n(name)].to(torch.float32).contiguous()
        self.proj = Linear(tensors[n("in")], self.ctx.num_sms)
        self.conv.load(tensors[n("conv")], tensors[n("conv.b")])
        self.dt_bias, self.a_log, self.skip, self.norm_w = f32("dt_bias"), f32("A_log"), f32("D"), f32("norm")
        self.o = Linear(tensors[n("o")], self.ctx.num_sms)

    def forward(self, h: torch.Tensor, step: StepContext, cache) -> torch.Tensor:
        conv_cache, state_cache = cache
        T, dev, I, C, GN = h.shape[0], h.device, self.inner, self.channels, self.G * self.N
        proj = self.proj(h, out_dtype=torch.float32)                     # [T, z | x B C | dt]
        xbc = torch.empty((T, C), dtype=torch.float32, device=dev)
        sizes = torch.empty((2, T, self.H), dtype=torch.float32, device=dev)     # step sizes, decays
        self.conv.run(proj[:, I: I + C], step, conv_cache, xbc, residual=False,
                      steps=(proj[:, I + C:], self.dt_bias, self.a_log, sizes[0], sizes[1]))
        x = xbc[:, :I]
        y = torch.empty((T, I), dtype=torch.float32, device=dev)
        K.head_scan(xbc[:, I + GN:], xbc[:, I: I + GN], x, sizes[1], 1.0, y, state_cache.state, step.cu_q, step.state_slots,
                    step.num_entries, self.H, self.N, self.vd, gain=sizes[0], key_heads=self.G)
        out = torch.empty((T, I), dtype=self.ctx.dtype, device=dev)
        K.part_norm_gate(y, proj[:, :I], self.norm_w, self.norm_groups, self.norm_eps, True, out, skip=(self.skip, x))
        return self.o(out, out_dtype=torch.float32)
