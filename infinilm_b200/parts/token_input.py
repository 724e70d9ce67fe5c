"""A layer's own input from its tokens: every layer owns some columns of a table with a row per token (`ModelSpec.token_table`);
at the layer's end they come into the residual stream through a gate that reads the stream,

    g = gelu_tanh(W_gate x) * e;   y = W_proj g;   x <- x + rms_norm(y) * w          (e: the layer's columns of the token's row)

x enters the gate as it stands in the stream, not normed. Tensors (under the part's prefix): gate [dim, hidden], proj [hidden, dim],
norm [hidden].
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from .base import Part
from .linear import Linear
from .spec import WeightSpec


class TokenInput(Part):
    """params: hidden, dim, offset (first of the layer's columns of the table), eps. `dim` is padded to a multiple of 8 inside (the
    products read rows 16 bytes at a time); the surplus is zero in both weights."""
    graph_safe = True

    def __init__(self, params, prefix, dtype):
        super().__init__(params, prefix, dtype)
        self.hidden, self.dim, self.offset, self.eps = int(params["hidden"]), int(params["dim"]), int(params["offset"]), float(params["eps"])
        if self.dim < 1:
            raise ValueError("token input: at least one column per layer")
        self.dim_pad = (self.dim + 7) // 8 * 8
        self.gate, self.proj = Linear(self.hidden, self.dim_pad, dtype), Linear(self.dim_pad, self.hidden, dtype)
        self.norm_w: Optional[torch.Tensor] = None

    def weight_specs(self) -> List[WeightSpec]:
        return [WeightSpec("gate", (self.dim, self.hidden)), WeightSpec("proj", (self.hidden, self.dim), init=("normal", 0.1)),
                WeightSpec("norm", (self.hidden,), "vector", ("ones_normal", 0.05))]

    def set_weights(self, t: Dict[str, torch.Tensor]) -> None:
        pad = self.dim_pad - self.dim
        self.gate.set(torch.nn.functional.pad(t["gate"], (0, 0, 0, pad)))
        self.proj.set(torch.nn.functional.pad(t["proj"], (0, pad)))
        self.norm_w = t["norm"].contiguous()

    def branch(self, x: torch.Tensor, table: torch.Tensor, ctx) -> torch.Tensor:
        """x: the residual stream's rows in the compute dtype; table: the token table's tensor. Returns y, before its norm."""
        T = x.shape[0]
        g = ctx.ws.rows("token_gated", T, self.dim_pad, self.dtype)
        if self.dtype == torch.bfloat16 and ops.skinny_ok(T, self.hidden):
            ops.gemm_skinny_gelu_row(x, self.gate.weight, ctx.token_ids, table, self.offset, self.dim, g)
        else:
            z = self.gate(x, ctx.ws.rows("token_gate", T, self.dim_pad, torch.float32), out_f32=True)
            ops.gelu_row(z, ctx.token_ids, table, self.offset, self.dim, g)
        return self.proj(g, ctx.ws.rows("token_branch", T, self.hidden, self.dtype))
