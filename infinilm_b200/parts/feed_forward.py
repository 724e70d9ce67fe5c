"""Dense feed-forwards. Without a gate: down(relu(up(x))^2). Gated: down(act(gate(x)) * up(x)), act SiLU (SwiGLU) or the tanh form of GELU; or, "clamped", with
g = min(gate(x), limit) and u = up(x) kept within -limit .. limit: down(g sigmoid(alpha g) (u + 1)).

Parity with InfiniLM: `csrc/layers/mlp/mlp.cpp:7-38` (gate and up as one product, `swiglu(up, gate)`,
then down), `csrc/layers/linear/fused_linear.cpp:152-158,177-185` (gate rows first, up rows second).
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import ops
from .base import FeedForward, register_part
from .linear import Linear
from .spec import WeightSpec


class SwiGLU(FeedForward):
    """params: hidden, intermediate, bias, out_scale; activation ("silu", the default, or "gelu_tanh": the gate's function; or
    "clamped" with limit and alpha);
    names (local tensor names of the three weights, default gate_proj.weight / up_proj.weight / down_proj.weight)."""
    graph_safe = True
    ACTIVATIONS = {"silu": ops.ACT_SILU, "gelu_tanh": ops.ACT_GELU_TANH, "clamped": ops.ACT_CLAMPED}

    def __init__(self, params, prefix, dtype):
        super().__init__(params, prefix, dtype)
        self.hidden, self.inter = int(params["hidden"]), int(params["intermediate"])
        self.bias = bool(params.get("bias", False))
        act = str(params.get("activation", "silu"))
        if act not in self.ACTIVATIONS:
            raise ValueError(f"gated feed-forward: activation {act!r} is not one of {', '.join(self.ACTIVATIONS)}")
        self.act = self.ACTIVATIONS[act]
        self.act_params = (float(params["limit"]), float(params["alpha"])) if self.act == ops.ACT_CLAMPED else None
        if self.act_params is not None and not self.act_params[0] > 0.0:
            raise ValueError("gated feed-forward: the clamped gate's limit must be positive")
        names = params.get("names") or {}
        self.n_gate, self.n_up, self.n_down = (str(names.get(k, d)) for k, d in
                                               (("gate", "gate_proj.weight"), ("up", "up_proj.weight"), ("down", "down_proj.weight")))
        if self.bias and names:
            raise ValueError("gated feed-forward: biases go with the default tensor names")
        self.gate_up = Linear(self.hidden, 2 * self.inter, dtype)
        self.down = Linear(self.inter, self.hidden, dtype, alpha=float(params.get("out_scale", 1.0)))

    def weight_specs(self) -> List[WeightSpec]:
        specs = [WeightSpec(self.n_gate, (self.inter, self.hidden)), WeightSpec(self.n_up, (self.inter, self.hidden)),
                 WeightSpec(self.n_down, (self.hidden, self.inter))]
        if self.bias:
            specs += [WeightSpec("gate_proj.bias", (self.inter,), "vector"), WeightSpec("up_proj.bias", (self.inter,), "vector"),
                      WeightSpec("down_proj.bias", (self.hidden,), "vector")]
        return specs

    def set_weights(self, t: Dict[str, torch.Tensor]) -> None:
        w = torch.cat([t[self.n_gate], t[self.n_up]], dim=0)
        b = torch.cat([t["gate_proj.bias"].float(), t["up_proj.bias"].float()]) if self.bias else None
        self.gate_up.set(w, b)
        self.down.set(t[self.n_down], t.get("down_proj.bias"))

    def accepts_normed(self, T):
        return self.dtype == torch.bfloat16 and ops.skinny_ok(T, self.hidden)

    def fuses_tail(self, T):
        return self.dtype == torch.bfloat16 and ops.skinny_ok(T, self.hidden) and ops.skinny_resid_ok(T, self.inter, self.hidden)

    def forward(self, x, ctx, tail=None):
        T = x.shape[0]
        if self.dtype == torch.bfloat16 and ops.skinny_ok(T, self.hidden):
            # decode: gate and up rows streamed together, SiLU(gate)*up in the epilogue
            act = ctx.ws.rows("ffn_act", T, self.inter, self.dtype)
            if isinstance(x, ops.NormedInput):
                ops.gemm_skinny(x.xw, self.gate_up.weight, act, 1.0, self.gate_up.bias, glu=self.act, norm_in=x, act_params=self.act_params)
            else:
                ops.gemm_skinny(x, self.gate_up.weight, act, 1.0, self.gate_up.bias, glu=self.act, act_params=self.act_params)
            if tail is not None:                  # down adds into the residual and prepares the next norm itself
                return ops.gemm_skinny_resid(act, self.down.weight, self.down.alpha, self.down.bias, tail.resid, tail.scale,
                                             tail.norm.weight, tail.norm.eps,
                                             ctx.ws.rows("xw_ffn", T, self.hidden, self.dtype),
                                             ctx.ws.rows("sumsq_ffn", T, (self.hidden + 15) // 16, torch.float32))
            return self.down(act, ctx.ws.rows("ffn_branch", T, self.hidden, self.dtype))
        act = ctx.ws.rows("ffn_act", T, self.inter, self.dtype)
        if self.dtype == torch.bfloat16 and ops.mid_ok(T, self.hidden):
            # 17..128 rows: gate and up on the tcgen05 tensor cores as two accumulators in the same lanes, SiLU(gate)*up in
            # the epilogue (measured against the library product followed by the SwiGLU kernel at 8B sizes: 44.6 against
            # 48.4 us at 32 rows, 47.6 against 49.9 at 64, 52.5 against 57.6 at 128)
            ops.gemm_mid(x, self.gate_up.weight, act, 1.0, self.gate_up.bias, glu=self.act, act_params=self.act_params)
            return self.down(act, ctx.ws.rows("ffn_branch", T, self.hidden, self.dtype))
        gu = self.gate_up(x, ctx.ws.rows("gate_up", T, 2 * self.inter, self.dtype))
        ops.swiglu(gu, act, self.act, self.act_params)
        return self.down(act, ctx.ws.rows("ffn_branch", T, self.hidden, self.dtype))


class SquaredReLU(FeedForward):
    """down(relu(up(x))^2). params: hidden, intermediate, names (local tensor names of the two weights, default up_proj.weight /
    down_proj.weight)."""
    graph_safe = True

    def __init__(self, params, prefix, dtype):
        super().__init__(params, prefix, dtype)
        self.hidden, self.inter = int(params["hidden"]), int(params["intermediate"])
        names = params.get("names") or {}
        self.n_up, self.n_down = str(names.get("up", "up_proj.weight")), str(names.get("down", "down_proj.weight"))
        self.up, self.down = Linear(self.hidden, self.inter, dtype), Linear(self.inter, self.hidden, dtype)

    def weight_specs(self) -> List[WeightSpec]:
        return [WeightSpec(self.n_up, (self.inter, self.hidden)), WeightSpec(self.n_down, (self.hidden, self.inter))]

    def set_weights(self, t: Dict[str, torch.Tensor]) -> None:
        self.up.set(t[self.n_up])
        self.down.set(t[self.n_down])

    def accepts_normed(self, T):
        return self.dtype == torch.bfloat16 and ops.skinny_ok(T, self.hidden)

    def fuses_tail(self, T):
        return self.dtype == torch.bfloat16 and ops.skinny_ok(T, self.hidden) and ops.skinny_resid_ok(T, self.inter, self.hidden)

    def forward(self, x, ctx, tail=None):
        T = x.shape[0]
        act = ctx.ws.rows("ffn_act", T, self.inter, self.dtype)
        if self.dtype == torch.bfloat16 and ops.skinny_ok(T, self.hidden):      # the activation in the product's epilogue
            normed = isinstance(x, ops.NormedInput)
            ops.gemm_skinny(x.xw if normed else x, self.up.weight, act, glu=ops.ACT_RELU2, norm_in=x if normed else None)
        elif self.dtype == torch.bfloat16 and ops.mid_ok(T, self.hidden):
            ops.gemm_mid(x, self.up.weight, act, glu=ops.ACT_RELU2)
        else:
            self.up(x, act)
            ops.relu2(act, act)
        if tail is not None:                      # down adds into the residual and prepares the next norm itself
            return ops.gemm_skinny_resid(act, self.down.weight, self.down.alpha, self.down.bias, tail.resid, tail.scale,
                                         tail.norm.weight, tail.norm.eps, ctx.ws.rows("xw_ffn", T, self.hidden, self.dtype),
                                         ctx.ws.rows("sumsq_ffn", T, (self.hidden + 15) // 16, torch.float32))
        return self.down(act, ctx.ws.rows("ffn_branch", T, self.hidden, self.dtype))


register_part("feed_forward", "swiglu", SwiGLU)
register_part("feed_forward", "squared_relu", SquaredReLU)
