"""Dense feed-forwards: the gated one, ``down( silu(gate(x)) * up(x) )``, and one without a gate (``PlainMLP``).

gate and up are stacked once at load into one ``[2I, h]`` matrix whose rows are (gate_j, up_j) pairs, so
that one product feeds the gate (the reference stacks them as two halves and runs the gate as its own
kernel: crates/layers/src/nn.rs:288-311,373-381).  With the pairs in neighbouring rows the decode
product applies the gate in its epilogue; prompts run the product and then the gate kernel."""
from __future__ import annotations

from typing import Dict, List, Optional

import math

import torch

from .base import FEED_FORWARDS, FeedForward
from .linear import Linear
from .spec import TensorDecl


@FEED_FORWARDS.register("none")
class NoFeedForward(FeedForward):
    """A layer without a feed-forward: arrangements that know of it (``absent``) skip the branch."""
    absent = True

    def forward(self, x, ctx=None, sink=None):
        raise RuntimeError("this layer has no feed-forward")


@FEED_FORWARDS.register("gated_mlp")
@FEED_FORWARDS.register("swiglu")
class SwiGLU(FeedForward):
    """``down( act(gate(x)) * up(x) )``.  params: ``intermediate_size``, optional ``activation`` (silu, the default;
    gelu_tanh, relu, relu2), ``out_float32`` (the down projection's result stays 32-bit, for an arrangement that norms
    it before it joins the stream) and tensor names ``gate_proj``, ``up_proj``, ``down_proj``."""

    def __init__(self, params, env, prefix=""):
        super().__init__(params, env, prefix)
        self.hidden = env.hidden_size
        self.inter = int(params["intermediate_size"])
        self.activation = str(params.get("activation", "silu"))
        self.out_float32 = bool(params.get("out_float32", False))
        from ..kernels.ops import GATE_ACTIVATIONS
        if self.activation not in GATE_ACTIVATIONS:
            raise ValueError(f"gated feed-forward: unknown activation {self.activation!r} ({', '.join(GATE_ACTIVATIONS)})")
        n = lambda key, default: prefix + params.get(key, default)
        self.names = {"g": n("gate_proj", "gate_proj.weight"), "u": n("up_proj", "up_proj.weight"),
                      "d": n("down_proj", "down_proj.weight")}
        self.gate_up: Optional[Linear] = None
        self.down: Optional[Linear] = None

    def declare(self) -> List[TensorDecl]:
        return [TensorDecl(self.names["g"], (self.inter, self.hidden)),
                TensorDecl(self.names["u"], (self.inter, self.hidden)),
                TensorDecl(self.names["d"], (self.hidden, self.inter))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        g, u = tensors[self.names["g"]], tensors[self.names["u"]]
        dt = torch.float32 if torch.float32 in (g.dtype, u.dtype) else g.dtype
        # row 2j = gate_j, row 2j + 1 = up_j
        self.gate_up = Linear(torch.stack([g.to(dt), u.to(dt)], dim=1).reshape(2 * self.inter, self.hidden))
        self.down = Linear(tensors[self.names["d"]])

    def kernel_libraries(self):
        return ["elementwise"] + self.gate_up.kernel_libraries() + self.down.kernel_libraries()

    def takes_half_normed(self, rows: int) -> bool:
        return (self.activation == "silu" and self.gate_up.fuses_norm(rows, self.env.act_dtype)
                and self.gate_up.out_features % 2 == 0)

    def adds_into_residual(self, rows: int) -> bool:
        return self.down.fuses_norm(rows, self.env.act_dtype)

    def forward(self, x, ctx=None, sink=None):
        act = self.gate_up.gated_pairs(x, self.activation)
        if sink is not None:                               # (residual, the norm behind this feed-forward)
            return self.down.into_residual(act, sink[0], sink[1])
        return self.down(act, out_dtype=torch.float32 if self.out_float32 else None)


@FEED_FORWARDS.register("plain_mlp")
class PlainMLP(FeedForward):
    """``down( act(up(x)) )``, no gate.  params: ``intermediate_size``, ``activation`` (relu, relu2, silu, gelu_tanh, or
    xielu, whose two learned numbers are the tensor ``act``: with a_pos = softplus(act[0]) and a_neg = 1/2 + softplus(act[1]),
    ``z / 2 + a_pos z^2`` above zero and ``z / 2 + a_neg (exp(z) - 1 - z)`` below), tensor names ``up_proj``, ``down_proj``,
    ``act``.  The activation is 32-bit, in the epilogue of the up product where that is this package's own."""

    def __init__(self, params, env, prefix=""):
        super().__init__(params, env, prefix)
        self.hidden = env.hidden_size
        self.inter = int(params["intermediate_size"])
        self.activation = str(params.get("activation", "relu2"))
        from ..kernels.gemm_ops import UNARY
        if self.activation not in UNARY:
            raise ValueError(f"feed-forward: unknown activation {self.activation!r}")
        n = lambda key, default: prefix + params.get(key, default)
        self.names = {"u": n("up_proj", "up_proj.weight"), "d": n("down_proj", "down_proj.weight"), "a": n("act", "act")}
        self.up: Optional[Linear] = None
        self.down: Optional[Linear] = None

    def declare(self) -> List[TensorDecl]:
        d = [TensorDecl(self.names["u"], (self.inter, self.hidden)), TensorDecl(self.names["d"], (self.hidden, self.inter))]
        if self.activation == "xielu":
            d.append(TensorDecl(self.names["a"], (2,)))
        return d

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.up, self.down = Linear(tensors[self.names["u"]]), Linear(tensors[self.names["d"]])
        self.act = self.activation
        if self.activation == "xielu":
            p, q = (float(v) for v in tensors[self.names["a"]].double().cpu())
            softplus = lambda v: max(v, 0.0) + math.log1p(math.exp(-abs(v)))
            self.act = ("xielu", softplus(p), 0.5 + softplus(q))

    def kernel_libraries(self):
        return ["moe"] + self.up.kernel_libraries() + self.down.kernel_libraries()

    def forward(self, x, ctx=None, sink=None):
        return self.down(self.up.activated(x, self.act))
