"""A layer's own small input per token, joined to the stream behind the layer's sublayers:

    e = table[token][at : at + dim];   y = W_proj (gelu_tanh(W_gate x) * e);   x <- x + y / rms(y) * w

The table is one tensor for all layers, a layer's part of a token's row starting at ``index * dim``.  The token ids are
the step's (``StepContext.token_ids``), placeholders of the last step's samples included."""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import BuildEnv, Part, StepContext
from .linear import Linear
from .norm import RMSNorm
from .spec import TensorDecl


class TokenSide(Part):
    """params: ``dim``, ``index`` (the layer's place among ``layers``), ``vocab_size``, ``eps``, ``table`` (tensor name, no
    prefix), ``gate_proj``, ``out_proj``, ``norm`` (tensor names after the layer's prefix)."""

    def __init__(self, params, env: BuildEnv, prefix=""):
        super().__init__(params, env, prefix)
        p = self.params
        self.dim, self.index, self.layers = int(p["dim"]), int(p["index"]), int(p["layers"])
        if self.dim <= 0 or not (0 <= self.index < self.layers):
            raise ValueError("token side: dim must be positive and the layer one of its layers")
        self.vocab = int(p["vocab_size"])
        self.names = {"table": p["table"], "gate": prefix + p["gate_proj"], "proj": prefix + p["out_proj"]}
        self.norm = RMSNorm({"size": env.hidden_size, "eps": float(p["eps"]), "weight": p["norm"]}, env, prefix)

    def declare(self) -> List[TensorDecl]:
        h = self.env.hidden_size
        return [TensorDecl(self.names["table"], (self.vocab, self.layers * self.dim)), TensorDecl(self.names["gate"], (self.dim, h)),
                TensorDecl(self.names["proj"], (h, self.dim))] + self.norm.declare()

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors[self.names["table"]]
        self.gate, self.proj = Linear(tensors[self.names["gate"]]), Linear(tensors[self.names["proj"]])
        self.norm.bind(tensors)

    def kernel_libraries(self):
        return ["token_side"] + self.gate.kernel_libraries() + self.proj.kernel_libraries()

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        """x [T, h], the stream in the activation type -> y [T, h], not normed yet."""
        from ..kernels import stream_ops
        if ctx.token_ids is None:
            raise RuntimeError("the token side needs the step's token ids (StepContext.token_ids)")
        u = stream_ops.token_gate(self.gate(x), ctx.token_ids, self.table, self.index * self.dim, ctx.prev_tokens)
        return self.proj(u)
