"""Dense gated feed-forward: down( silu(gate(x)) * up(x) ), or with the tanh form of gelu in place of silu
(crates/infer-worker/src/components/ffn_dense.rs:26-33,76-115).  gate and up are fused by
rows into one matrix, gate rows first (crates/infer-worker/src/models/loader.rs:543-571)."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..ops import kernels as K
from .base import FeedForward, ParamDecl, StepContext, register_feed_forward
from .linear import Linear


@register_feed_forward("swiglu")
class SwiGLU(FeedForward):
    """params: hidden_size, intermediate_size, output ("float32": the result leaves the down projection in
    32-bit, default the activation dtype), activation ("silu", the default, or "gelu_tanh"), gate_name / up_name /
    down_name (tensor names, default "gate_proj.weight" and so on)."""

    def __init__(self, params):
        super().__init__(params)
        self.hidden = int(params["hidden_size"])
        self.inter = int(params["intermediate_size"])
        self.out_fp32 = str(params.get("output", "")) == "float32"
        self.activation = str(params.get("activation", "silu"))
        if self.activation not in ("silu", "gelu_tanh"):
            raise ValueError(f"gated feed-forward activation {self.activation!r}: known are 'silu' and 'gelu_tanh'")
        self.names = {k: str(params.get(k + "_name", k + "_proj.weight")) for k in ("gate", "up", "down")}
        self.gate_up: Optional[Linear] = None
        self.down: Optional[Linear] = None

    def param_decls(self) -> Dict[str, ParamDecl]:
        return {self.names["gate"]: ParamDecl((self.inter, self.hidden)),
                self.names["up"]: ParamDecl((self.inter, self.hidden)),
                self.names["down"]: ParamDecl((self.hidden, self.inter))}

    adds_to_residual = True

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        g, u = tensors[self.names["gate"]], tensors[self.names["up"]]
        dt = torch.float32 if torch.float32 in (g.dtype, u.dtype) else g.dtype
        sms = self.ctx.num_sms
        # bf16: rows alternate gate_j, up_j so that the product's epilogue can form
        # act(gate) * up; fp32: gate rows first, then up rows, for the separate kernel
        self.paired = dt == torch.bfloat16 and self.hidden % 8 == 0 and g.is_cuda
        if self.paired:
            self.gate_up = Linear(torch.stack([g.to(dt), u.to(dt)], dim=1).reshape(2 * self.inter, self.hidden), sms)
        else:
            self.gate_up = Linear(torch.cat([g.to(dt), u.to(dt)], dim=0), sms)
        self.down = Linear(tensors[self.names["down"]], sms)

    def forward(self, x: torch.Tensor, step: StepContext, residual: Optional[torch.Tensor] = None):
        """Returns the sublayer's output, or None when it was added into `residual`."""
        gelu = self.activation == "gelu_tanh"
        m = self.gate_up.gated_pairs(x, gelu) if self.paired else None
        if m is None:
            gu = self.gate_up(x, out_dtype=self.ctx.dtype)
            if self.paired:                               # the fused path refused this input
                gu = torch.cat([gu[:, 0::2], gu[:, 1::2]], dim=1).contiguous()
            m = torch.empty((x.shape[0], self.inter), dtype=self.ctx.dtype, device=x.device)
            K.silu_mul(gu, m, gelu)
        if residual is not None and self.down.add_into(m, residual):
            return None
        return self.down(m, out_dtype=torch.float32 if self.out_fp32 else self.ctx.dtype)


_ACTIVATIONS = {"gelu": K.ACT_GELU_ERF, "gelu_erf": K.ACT_GELU_ERF, "tanh": K.ACT_TANH, "gelu_tanh": K.ACT_GELU_TANH,
                "relu_squared": K.ACT_RELU_SQUARED, "silu": K.ACT_SILU}


@register_feed_forward("dense_mlp")
class DenseMLP(FeedForward):
    """down( act(up(x)) ) without a gate.  params: hidden_size, intermediate_size, activation
    ("gelu": with erf; "gelu_tanh"; "tanh"; "relu_squared": max(z, 0)^2; "silu"), up_name / down_name (tensor names, default
    "up_proj.weight" / "down_proj.weight"), output ("float32": the result leaves the down projection in
    32-bit).  The activation is computed in fp32; the square of relu in the bfloat16 engine inside the
    up product's epilogue, from the unrounded sums."""

    def __init__(self, params):
        super().__init__(params)
        self.hidden = int(params["hidden_size"])
        self.inter = int(params["intermediate_size"])
        act = str(params.get("activation", "gelu"))
        if act not in _ACTIVATIONS:
            raise ValueError(f"activation {act!r}: known are {sorted(_ACTIVATIONS)}")
        self.act = _ACTIVATIONS[act]
        self.up_name = str(params.get("up_name", "up_proj.weight"))
        self.down_name = str(params.get("down_name", "down_proj.weight"))
        self.out_fp32 = str(params.get("output", "")) == "float32"
        self.up: Optional[Linear] = None
        self.down: Optional[Linear] = None

    def param_decls(self) -> Dict[str, ParamDecl]:
        return {self.up_name: ParamDecl((self.inter, self.hidden)),
                self.down_name: ParamDecl((self.hidden, self.inter))}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.up = Linear(tensors[self.up_name], self.ctx.num_sms)
        self.down = Linear(tensors[self.down_name], self.ctx.num_sms)

    def forward(self, x: torch.Tensor, step: StepContext, residual: Optional[torch.Tensor] = None):
        u = self.up.relu_squared(x) if self.act == K.ACT_RELU_SQUARED and self.ctx.dtype == torch.bfloat16 else None
        if u is None:                                     # other activations, the 32-bit engine, inputs the fused path refuses
            u = self.up(x, out_dtype=self.ctx.dtype)
            K.activation(u, u, self.act)
        if residual is not None and self.down.add_into(u, residual):
            return None
        return self.down(u, out_dtype=torch.float32 if self.out_fp32 else self.ctx.dtype)
