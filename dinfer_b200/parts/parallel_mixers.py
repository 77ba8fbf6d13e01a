"""Two mixers side by side: both read the same rows, each output is divided by its own root mean square over the
model width and multiplied by a weight of its own, and the result is the weighted sum of the two (half the sum:
their mean).  The two keep what they keep independently: the pair's cache need is the list of theirs (at most one
paged cache and one fixed-size state between them), and both get the entry's binding.

With ``scales`` the two are not normed: the result is ``scale_left * left + scale_right * right``.  Both mixers then have
open ends (``Mixer.open_ends``): one product of the stacked input matrices feeds both, and one product of both output
matrices side by side, over rows that hold both mixers' results, makes the sum; the scales are folded into the mixers."""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import MIXERS, BuildEnv, CacheBinding, Mixer, NormedBranches, StepContext, build_part, split_needs
from .linear import Linear
from .spec import PartSpec, TensorDecl


@MIXERS.register("parallel_mixers")
class ParallelMixers(Mixer):
    """params: ``left`` / ``right`` (PartSpecs of two mixers; their tensor names follow the pair's prefix),
    ``left_out`` / ``right_out`` (tensor names of the per-channel weights behind each branch's norm), ``eps``,
    ``coef`` (0.5: the mean); or ``scales`` = (left, right) instead of the last three."""

    def __init__(self, params, env: BuildEnv, prefix=""):
        super().__init__(params, env, prefix)
        p = self.params
        self.left: Mixer = build_part(MIXERS, p["left"], env, prefix)
        self.right: Mixer = build_part(MIXERS, p["right"], env, prefix)
        self.scales = tuple(float(v) for v in p["scales"]) if p.get("scales") is not None else None
        if self.scales is not None and (self.left.open_ends() is None or self.right.open_ends() is None):
            raise ValueError("parallel_mixers: a weighted sum needs two mixers with open ends")
        self.eps = float(p.get("eps", 0.0))
        self.coef = float(p.get("coef", 0.5))
        self.names = (prefix + p.get("left_out", "left.out"), prefix + p.get("right_out", "right.out"))
        split_needs(self.cache_need())                     # refuses two of a kind

    @property
    def graph_capturable(self):
        return all(m.cache_need() is None or getattr(m, "graph_capturable", False) or
                   split_needs(m.cache_need())[1] is None for m in (self.left, self.right))

    def declare(self) -> List[TensorDecl]:
        h = self.env.hidden_size
        if self.scales is not None:
            return self.left.declare() + self.right.declare()
        return (self.left.declare() + self.right.declare()
                + [TensorDecl(self.names[0], (h,), init="ones"), TensorDecl(self.names[1], (h,), init="ones")])

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        if self.scales is not None:
            return self._bind_stacked(tensors)
        self.left.bind(tensors)
        self.right.bind(tensors)
        self.left_w, self.right_w = (tensors[n].contiguous() for n in self.names)
        if self.left_w.dtype != self.right_w.dtype:
            self.left_w, self.right_w = self.left_w.float(), self.right_w.float()

    def _bind_stacked(self, tensors: Dict[str, torch.Tensor]) -> None:
        """The two products.  Each mixer's part of the projected rows and of the result rows starts at a multiple of 8
        columns (zeros between), for vector loads and TMA."""
        up8 = lambda n: (n + 7) // 8 * 8
        rows, cols = [], []
        for m, scale in zip((self.left, self.right), self.scales):
            w, o = m.input_rows(tensors), m.output_columns(tensors)
            n_in, n_out = m.open_ends()
            if w.shape[0] != n_in or o.shape[1] != n_out:
                raise ValueError("parallel_mixers: a mixer's matrices are not as wide as its open ends")
            rows += [w, w.new_zeros((up8(n_in) - n_in, w.shape[1]))]
            cols += [o, o.new_zeros((o.shape[0], up8(n_out) - n_out))]
            m.bind_inner(tensors, scale)
        def one(parts, dim):
            dt = torch.float32 if any(t.dtype == torch.float32 for t in parts) else parts[0].dtype
            return Linear(torch.cat([t.to(dt) for t in parts], dim=dim))
        self.proj, self.o = one(rows, 0), one(cols, 1)
        (a_in, a_out), (b_in, b_out) = self.left.open_ends(), self.right.open_ends()
        self.in_at, self.out_at = up8(a_in), up8(a_out)
        self.left_out, self.right_out = a_out, b_out
        self.padded = up8(a_out) != a_out or up8(b_out) != b_out

    def cache_need(self):
        return [n for m in (self.left, self.right) for n in split_needs(m.cache_need()) if n is not None]

    def kernel_libraries(self):
        if self.scales is not None:
            return (self.left.kernel_libraries() + self.right.kernel_libraries() + self.proj.kernel_libraries()
                    + self.o.kernel_libraries())
        return ["norm"] + self.left.kernel_libraries() + self.right.kernel_libraries()

    def takes_half_normed(self, rows: int) -> bool:
        return self.scales is not None and self.proj.fuses_norm(rows, self.env.act_dtype)

    def adds_into_residual(self, rows: int) -> bool:
        return self.scales is not None and self.o.fuses_norm(rows, self.env.act_dtype)

    def forward(self, x, ctx: StepContext, cache: CacheBinding, sink=None):
        if self.scales is not None:
            P = self.proj(x, out_dtype=torch.float32)
            make = torch.zeros if self.padded else torch.empty
            y = make((P.shape[0], self.o.in_features), dtype=self.env.act_dtype, device=P.device)
            self.left.mix(P[:, :self.in_at], y[:, :self.left_out], ctx, cache)
            self.right.mix(P[:, self.in_at:], y[:, self.out_at:self.out_at + self.right_out], ctx, cache)
            if sink is not None:                           # (residual, the norm behind this mixer)
                return self.o.into_residual(y, sink[0], sink[1])
            return self.o(y)
        a = self.left.forward(x, ctx, cache)
        b = self.right.forward(x, ctx, cache)
        return NormedBranches([(a, self.left_w), (b, self.right_w)], self.coef, self.eps)
