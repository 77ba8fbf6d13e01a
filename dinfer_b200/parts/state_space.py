"""A state-space mixer with one decay per head and token (Mamba-2's form).  One product gives a token's row
``[z: inner | x: inner | B: G N | C: G N | dt: H]`` with ``inner = H P``; x, B and C pass a short causal convolution per
channel (with a bias) and silu.  Per head (B and C of its group) a matrix S [N, P] in 32-bit is carried from token to token:

    dt = softplus(dt + dt_bias),   S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t

The heads' y times ``silu(z)`` is RMS-normed in equal parts of the row, multiplied by a weight and projected.

Data flow of one step (prompt portions and decoded tokens alike):
  P = x W_in^T                          its result stays 32-bit
  y = state_space(P, state)             32-bit; single tokens in one kernel, portions in chunks side by side
  o = norm(y * silu(z))                 one kernel, which also moves the convolution's inputs into the state
  out = o W_o^T
What a request keeps is one row of a fixed-size state: S of every head, then the convolution's last ``taps - 1`` inputs.
Slots and fresh flags are read from the device only, so steps replay as CUDA graphs.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import state_ops
from .base import MIXERS, BuildEnv, CacheBinding, Mixer, StateNeed, StepContext
from .linear import Linear
from .spec import TensorDecl


@MIXERS.register("state_space")
class StateSpace(Mixer):
    """params: ``num_heads``, ``value_dim`` (P), ``state_dim`` (N), ``groups`` (heads share B and C), ``conv`` (taps),
    ``norm_parts``, ``eps`` (of the output norm), ``out_float32``, and the tensor names ``in_proj``, ``conv_weight``,
    ``conv_bias``, ``dt_bias``, ``A_log``, ``D``, ``norm``, ``o_proj``."""

    graph_capturable = True

    def __init__(self, params, env: BuildEnv, prefix=""):
        super().__init__(params, env, prefix)
        p = self.params
        self.hidden = env.hidden_size
        self.H, self.P, self.N = int(p["num_heads"]), int(p["value_dim"]), int(p["state_dim"])
        self.G, self.taps, self.parts = int(p.get("groups", 1)), int(p["conv"]), int(p.get("norm_parts", 1))
        self.eps = float(p["eps"])
        self.out_float32 = bool(p.get("out_float32", False))
        if min(self.H, self.P, self.N, self.G, self.taps, self.parts) <= 0 or self.H % self.G or (self.H * self.P) % self.parts:
            raise ValueError(f"state_space: {self.H} heads of {self.N} x {self.P} in {self.G} groups, {self.taps} taps, "
                             f"{self.parts} norm parts")
        n = lambda key, default: prefix + p.get(key, default)
        self.names = {"in": n("in_proj", "in"), "conv": n("conv_weight", "conv"), "conv_b": n("conv_bias", "conv.b"),
                      "dt_bias": n("dt_bias", "dt_bias"), "A_log": n("A_log", "A_log"), "D": n("D", "D"),
                      "norm": n("norm", "norm"), "o": n("o_proj", "o")}
        self.inner = self.H * self.P
        self.channels = self.inner + 2 * self.G * self.N
        self.state_size = self.H * self.N * self.P
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None

    def declare(self) -> List[TensorDecl]:
        h, N = self.hidden, self.names
        return [TensorDecl(N["in"], (self.inner + self.channels + self.H, h)), TensorDecl(N["conv"], (self.channels, self.taps)),
                TensorDecl(N["conv_b"], (self.channels,)), TensorDecl(N["dt_bias"], (self.H,)), TensorDecl(N["A_log"], (self.H,)),
                TensorDecl(N["D"], (self.H,), init="ones"), TensorDecl(N["norm"], (self.inner,), init="ones"),
                TensorDecl(N["o"], (h, self.inner))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        w = tensors[self.names["in"]]
        pad = -w.shape[0] % 8                                # rows of whole 16-byte pieces
        self.proj = Linear(torch.cat([w, w.new_zeros((pad, w.shape[1]))]) if pad else w)
        self.o = Linear(tensors[self.names["o"]])
        self.bind_inner(tensors)

    # ---- between two products of another part (see Mixer.open_ends)
    def open_ends(self):
        return self.inner + self.channels + self.H, self.inner

    def input_rows(self, tensors) -> torch.Tensor:
        return tensors[self.names["in"]]

    def output_columns(self, tensors) -> torch.Tensor:
        return tensors[self.names["o"]]

    def bind_inner(self, tensors, scale: float = 1.0) -> None:
        f32 = lambda key: tensors[self.names[key]].to(torch.float32).contiguous()
        self.conv_w, self.conv_b, self.dt_bias, self.A_log, self.D = (f32(k) for k in ("conv", "conv_b", "dt_bias", "A_log", "D"))
        self.norm_w = f32("norm") * float(scale)             # the result is linear in the norm's weight

    def cache_need(self):
        n = self.state_size + (self.taps - 1) * self.channels
        return StateNeed(((n + 3) // 4 * 4,), torch.float32)     # rows of whole 16-byte pieces

    def kernel_libraries(self):
        return ["state_space"] + [n for l in (self.proj, self.o) if l is not None for n in l.kernel_libraries()]

    def mix(self, P, out, ctx: StepContext, cache: CacheBinding) -> None:
        B = ctx.cu_seqlens.numel() - 1
        slots, fresh = ctx.state_slots[:B], ctx.state_fresh[:B]
        sizes = (self.H, self.G, self.N, self.P, self.taps)
        y = state_ops.state_space(P, self.conv_w, self.conv_b, self.dt_bias, self.A_log, self.D, cache.state, ctx.cu_seqlens,
                                  slots, fresh, *sizes, any_single=ctx.any_decode, any_portion=ctx.any_prefill,
                                  max_q_len=ctx.max_q_len)
        state_ops.state_space_post(y, P, self.norm_w, self.eps, self.parts, out, cache.state, ctx.cu_seqlens, slots, fresh, *sizes)

    def forward(self, x, ctx: StepContext, cache: CacheBinding):
        P = self.proj(x, out_dtype=torch.float32)
        y = torch.empty((x.shape[0], self.inner), dtype=self.env.act_dtype, device=x.device)
        self.mix(P, y, ctx, cache)
        return self.o(y, out_dtype=torch.float32 if self.out_float32 else None)
