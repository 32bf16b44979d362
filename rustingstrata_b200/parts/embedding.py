"""Token embedding (row lookup without scale, src/model.rs:334-339) and the output head
(final norm is a norm part; the head is one matrix, the token table itself when tied,
src/model.rs:602-607)."""
from __future__ import annotations

from ..kernels import ops
from .base import Part
from .registry import register_part
from .spec import TensorNeed


@register_part("embedding", "token_table")
class TokenEmbedding(Part):
    """params: vocab, width, norm_eps (with a norm).  tensors: weight, and norm [width] for a model whose stream starts as the
    RMS norm of the token's row."""
    chain_safe = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.vocab = int(spec.params["vocab"])
        self.width = int(spec.params["width"])
        self.norm_eps = float(spec.params["norm_eps"]) if "norm" in spec.tensors else 0.0
        self.weight = self.norm_weight = None

    def tensor_needs(self):
        needs = {self.spec.tensors["weight"]: TensorNeed((self.vocab, self.width), "embedding")}
        if "norm" in self.spec.tensors:
            needs[self.spec.tensors["norm"]] = TensorNeed((self.width,), "norm")
        return needs

    def load(self, tensors):
        self.weight = tensors[self.spec.tensors["weight"]]
        if "norm" in self.spec.tensors:
            self.norm_weight = tensors[self.spec.tensors["norm"]].contiguous()

    def forward(self, ctx, residual):
        if self.norm_weight is not None:
            ops.embed_rmsnorm(self.weight, ctx.token_ids, self.norm_weight, self.norm_eps, residual, ctx.n_tokens, ctx.status)
            return
        ops.embed(self.weight, ctx.token_ids, residual[: ctx.n_tokens], ctx.status)


@register_part("head", "linear")
class LinearHead(Part):
    """params: vocab, width, scale (default 1: the logits are multiplied by it, in float32), softcap (None: none; else the
    logits z become softcap * tanh(z / softcap), in float32).  tensors: weight (names the token table when the head is
    tied, in which case both parts hold the same device tensor)."""
    chain_safe = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.vocab = int(spec.params["vocab"])
        self.width = int(spec.params["width"])
        self.scale = float(spec.params.get("scale", 1.0))
        self.softcap = float(spec.params["softcap"]) if spec.params.get("softcap") is not None else None
        if self.softcap is not None and not self.softcap > 0:
            raise ValueError(f"linear head: softcap must be positive, got {self.softcap}")
        self.weight = None

    def tensor_needs(self):
        return {self.spec.tensors["weight"]: TensorNeed((self.vocab, self.width), "embedding")}

    def load(self, tensors):
        self.weight = tensors[self.spec.tensors["weight"]]

    def forward(self, h, logits, n_rows, status=None):
        ops.linear(h, self.weight, logits, n_rows, status=status)
        if self.softcap is not None:
            ops.softcap_rows(logits, n_rows, self.softcap, self.scale)
        elif self.scale != 1.0:
            ops.scale_rows(logits, n_rows, self.scale)
