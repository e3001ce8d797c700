"""An input by token in every layer: a small vector of the token's own, gated by the stream and projected back to it.

    e = S[ids, column : column + dim];   out = W_proj ( gelu_tanh(W_gate x) * e )

S is one table of the model whose columns are dealt out to the layers, so every layer's part declares it under the same
name and all of them hold the one tensor; W_gate [dim, hidden] and W_proj [hidden, dim] are the layer's own.  The part
stands where a feed-forward does (the `side` of a block); the reference's block has no such sublayer
(crates/infer-worker/src/components/decoder_block.rs:13-32).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..ops import kernels as K
from .base import FeedForward, ParamDecl, StepContext, register_feed_forward
from .linear import Linear


@register_feed_forward("token_input")
class TokenInput(FeedForward):
    """params: hidden_size, vocab_size, dim, table_columns (columns of the table), column (this layer's first), table_name /
    gate_name / proj_name (tensor names).  x is the stream in the activation dtype; the result is fp32."""

    def __init__(self, params):
        super().__init__(params)
        p = params
        self.hidden, self.vocab, self.dim = int(p["hidden_size"]), int(p["vocab_size"]), int(p["dim"])
        self.columns, self.column = int(p["table_columns"]), int(p["column"])
        self.names = {k: str(p[k + "_name"]) for k in ("table", "gate", "proj")}
        if self.dim <= 0 or not 0 <= self.column <= self.columns - self.dim:
            raise ValueError(f"token_input: columns {self.column} to {self.column + self.dim} of a table of {self.columns}")

    def param_decls(self) -> Dict[str, ParamDecl]:
        return {self.names["table"]: ParamDecl((self.vocab, self.columns)),
                self.names["gate"]: ParamDecl((self.dim, self.hidden)),
                self.names["proj"]: ParamDecl((self.hidden, self.dim))}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors[self.names["table"]].contiguous()
        self.gate = Linear(tensors[self.names["gate"]], self.ctx.num_sms)
        self.proj = Linear(tensors[self.names["proj"]], self.ctx.num_sms)

    def forward(self, x: torch.Tensor, step: StepContext) -> torch.Tensor:
        z = self.gate(x, out_dtype=torch.float32)
        g = torch.empty((x.shape[0], self.dim), dtype=self.ctx.dtype, device=x.device)
        K.token_gate(z, step.token_ids, self.table, self.column, g)
        return self.proj(g, out_dtype=torch.float32)
