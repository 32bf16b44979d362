"""Gated feed-forward (SwiGLU): down(act(gate h) * (up h)), no biases.

Reference: src/model.rs:803-811,818-820 with silu(z) = z / (1 + exp(-z)) (src/ops.rs:14);
device: gate and up as one launch, then ``swiglu``, then down returned as a pending
residual (src/gpu_model.rs:3307-3328).  Here gate and up are one [2I, hidden] matrix,
and the down projection adds straight into the residual stream.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import FeedForward
from .registry import register_part
from .spec import TensorNeed


@register_part("feed_forward", "gated_mlp")
class GatedMLP(FeedForward):
    """params: hidden, intermediate, activation ("silu", the default, "gelu_tanh", or "clamped": with g = min(gate, limit) and
    u = up held in [-limit, limit], g sigmoid(alpha g) (u + 1)), and for "clamped" alpha and limit.
    tensors: gate_proj, up_proj, down_proj."""
    chain_safe = True
    joinable = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.hidden = int(spec.params["hidden"])
        self.inter = int(spec.params["intermediate"])
        act = spec.params.get("activation", "silu")
        if act not in ops.GATE_ACTIVATIONS:
            raise ValueError(f"gated_mlp: activation '{act}' has no kernel (known: {', '.join(sorted(ops.GATE_ACTIVATIONS))})")
        self.activation = act
        self.gate_constants = ops.NO_GATE_CONSTANTS
        if act == "clamped":
            self.gate_constants = (float(spec.params["alpha"]), float(spec.params["limit"]))
            if not self.gate_constants[1] > 0:
                raise ValueError(f"gated_mlp: the clamped gate's limit must be positive, got {self.gate_constants[1]}")
        self.row_cols = self.inter
        runtime.scratch("gate_up", runtime.max_batch_tokens, 2 * self.inter)
        runtime.scratch("ff_act", runtime.max_batch_tokens, self.inter)
        self.w_gate_up = self.w_down = None

    def tensor_needs(self):
        t = self.spec.tensors
        return {t["gate_proj"]: TensorNeed((self.inter, self.hidden)),
                t["up_proj"]: TensorNeed((self.inter, self.hidden)),
                t["down_proj"]: TensorNeed((self.hidden, self.inter))}

    def load(self, tensors):
        t = self.spec.tensors
        g, u = tensors[t["gate_proj"]], tensors[t["up_proj"]]
        if g.dtype != u.dtype:
            raise ValueError("gated_mlp: gate and up projections must share an element type")
        # bfloat16 engine with 16-byte aligned rows: gate and up rows alternate, so the product's epilogue
        # applies SiLU(gate)*up to neighbouring accumulator columns and the [T, 2I] intermediate never
        # reaches memory.  Otherwise [gate; up] stacked, followed by the separate activation kernel.
        self.fused = (g.dtype == torch.bfloat16 and self.runtime.dtype == torch.bfloat16 and self.hidden % 8 == 0)
        if self.fused:
            self.w_gate_up = torch.stack([g, u], dim=1).reshape(2 * self.inter, self.hidden).contiguous()
        else:
            self.w_gate_up = torch.cat([g, u], dim=0).contiguous()
        self.w_down = tensors[t["down_proj"]].contiguous()

    def forward_rows(self, h, rows, ctx):
        T = ctx.n_tokens
        if self.fused:
            ops.linear_swiglu(h, self.w_gate_up, rows, T, status=ctx.status, activation=self.activation, gate=self.gate_constants)
        else:
            gate_up = self.runtime.get_scratch("gate_up")[:, : 2 * self.inter]
            ops.linear(h, self.w_gate_up, gate_up, T)
            ops.silu_mul(gate_up, rows, T, self.activation, self.gate_constants)

    def forward(self, h, residual, ctx):
        T = ctx.n_tokens
        act = self.runtime.get_scratch("ff_act")[:, : self.inter]
        self.forward_rows(h, act, ctx)
        ctx.owed = ops.linear(act, self.w_down, residual, T, accumulate=not ctx.store_output, status=ctx.status,
                              may_defer=ctx.may_owe and not ctx.store_output)


@register_part("feed_forward", "activation_mlp")
class ActivationMLP(FeedForward):
    """down(act(up h)), no biases, with an activation that has learned numbers of its own.

    params: hidden, intermediate, activation: "xielu" (two numbers p, q per layer: for z > 0, softplus(p) z^2 + z / 2;
    for z <= 0, (1/2 + softplus(q)) (exp(z) - 1 - z) + z / 2) or "gelu_tanh" (none).
    tensors: up_proj, down_proj, and act [2] for xielu.  The activation's arithmetic is float32."""

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.hidden = int(spec.params["hidden"])
        self.inter = int(spec.params["intermediate"])
        self.activation = spec.params.get("activation", "xielu")
        if self.activation not in ops.ACTIVATIONS:
            raise ValueError(f"activation_mlp: activation '{self.activation}' has no kernel "
                             f"(known: {', '.join(sorted(ops.ACTIVATIONS))})")
        runtime.scratch("ff_act", runtime.max_batch_tokens, self.inter)
        self.act_params = None

    def tensor_needs(self):
        t = self.spec.tensors
        needs = {t["up_proj"]: TensorNeed((self.inter, self.hidden)), t["down_proj"]: TensorNeed((self.hidden, self.inter))}
        if self.activation == "xielu":
            needs[t["act"]] = TensorNeed((2,))
        return needs

    def load(self, tensors):
        t = self.spec.tensors
        self.w_up = tensors[t["up_proj"]].contiguous()
        self.w_down = tensors[t["down_proj"]].contiguous()
        if self.activation == "xielu":
            self.act_params = tensors[t["act"]].to(torch.float32).contiguous()

    def flops_per_token(self) -> float:
        return 4.0 * self.hidden * self.inter

    def forward(self, h, residual, ctx):
        T = ctx.n_tokens
        act = self.runtime.get_scratch("ff_act")[:, : self.inter]
        ops.linear(h, self.w_up, act, T, status=ctx.status)
        ops.activation(act, act, T, self.activation, self.act_params)
        ops.linear(act, self.w_down, residual, T, accumulate=not ctx.store_output, status=ctx.status)


@register_part("feed_forward", "token_gate")
class TokenGate(FeedForward):
    """What a layer takes from the token itself: W_out (gelu(W_gate h) * e), gelu in its tanh form and float32, e the columns
    [column, column + dim) of the token's row in a table.

    params: hidden, dim, vocab, column (first column of this layer's part of the table), table_width (columns of the table).
    tensors: gate_proj [dim, hidden], out_proj [hidden, dim], table [vocab, table_width]."""
    gathered = ("table",)         # a step reads rows of it, not the whole

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.dim, self.vocab = int(p["hidden"]), int(p["dim"]), int(p["vocab"])
        self.column, self.table_width = int(p["column"]), int(p["table_width"])
        if not 0 <= self.column <= self.table_width - self.dim:
            raise ValueError(f"token_gate: columns {self.column} to {self.column + self.dim} of a table of {self.table_width}")
        pad = (self.dim + 7) // 8 * 8
        self.pre_name, self.act_name = f"token_gate_pre_{pad}", f"token_gate_act_{pad}"
        runtime.scratch(self.pre_name, runtime.max_batch_tokens, pad, torch.float32)
        runtime.scratch(self.act_name, runtime.max_batch_tokens, pad)

    def tensor_needs(self):
        t = self.spec.tensors
        return {t["gate_proj"]: TensorNeed((self.dim, self.hidden)), t["out_proj"]: TensorNeed((self.hidden, self.dim)),
                t["table"]: TensorNeed((self.vocab, self.table_width), "embedding")}

    def load(self, tensors):
        t = self.spec.tensors
        self.w_gate = tensors[t["gate_proj"]].contiguous()
        self.w_out = tensors[t["out_proj"]].contiguous()
        self.table = tensors[t["table"]]

    def flops_per_token(self) -> float:
        return 4.0 * self.hidden * self.dim

    def forward(self, h, residual, ctx):
        rt, T = self.runtime, ctx.n_tokens
        pre = rt.get_scratch(self.pre_name, torch.float32)[:, : self.dim]
        act = rt.get_scratch(self.act_name)[:, : self.dim]
        ops.linear(h, self.w_gate, pre, T, status=ctx.status)
        ops.gelu_table_gate(pre, self.table, self.column, ctx.token_ids, act, T, ctx.status)
        ops.linear(act, self.w_out, residual, T, accumulate=not ctx.store_output, status=ctx.status)
