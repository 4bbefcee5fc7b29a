"""Two mixers side by side: both read the same input, and the result is a weighted sum of theirs.

The mixers are parts of the "mixer" family named by the spec; what a run keeps per sequence is what both keep (keys and
values of the one beside the state of the other, say), so `cache_need()` gives both needs and the cache hands a view
with the fields of both.

With `joined` the two input projections run as one product and the two output projections as another: both mixers read the
same rows, so their weights stand one below the other in front, and behind them scale_a Wa a + scale_b Wb b is the product
of [Wa | Wb] with the mixers' outputs side by side, each scaled (in fp32) before it is rounded.  A mixer that can be joined
has input_weight(), output_weight(), proj_width, out_width and core(proj, step, cache, out, scale).
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import kernels as K
from ..plan import PartPlan
from ..registry import part_class, register_part
from .base import Part
from .linear import Linear


@dataclass(frozen=True)
class ParallelMixersSpec:
    left: PartPlan                # family "mixer"
    right: PartPlan
    left_scale: float = 1.0
    right_scale: float = 1.0
    joined: bool = False          # one product in front of both mixers and one behind


@dataclass
class WeightedPair:
    """scale_a * a + scale_b * b, not summed yet: a block whose next kernel can take the sum (`sums_pairs`) gets this."""
    a: torch.Tensor
    scale_a: float
    b: torch.Tensor
    scale_b: float


@register_part("mixer", "parallel_mixers")
class ParallelMixers(Part):
    family = "mixer"
    roles = ()

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.gives_pairs = not spec.joined      # forward(..., as_pair=True) leaves the weighted sum to the caller's next kernel
        self.takes_pending_norm = self.adds_to_stream = spec.joined
        self.left = part_class("mixer", spec.left.kind)(spec.left.spec, spec.left.tensors, runtime)
        self.right = part_class("mixer", spec.right.kind)(spec.right.spec, spec.right.tensors, runtime)
        self.graph_safe = bool(getattr(self.left, "graph_safe", False) and getattr(self.right, "graph_safe", False))
        self.kernel_modules = tuple(sorted({"stream_ops", *getattr(self.left, "kernel_modules", ()),
                                            *getattr(self.right, "kernel_modules", ())}))

    def tensor_specs(self):
        return self.left.tensor_specs() + self.right.tensor_specs()

    def bind(self, loaded):
        self.left.bind(loaded)
        self.right.bind(loaded)
        if self.spec.joined:
            pair = (self.left, self.right)
            if len({w.dtype for m in pair for w in (m.input_weight(), m.output_weight())}) != 1:
                raise ValueError("the projections of two joined mixers are stored in different dtypes")
            self.proj = Linear(torch.cat([m.input_weight() for m in pair], dim=0).contiguous())
            self.o = Linear(torch.cat([m.output_weight() for m in pair], dim=1).contiguous())
            for m in pair:                      # their own copies are not read any more
                m.proj = m.o = None

    def prepare(self, max_positions: int) -> None:
        for m in (self.left, self.right):
            if hasattr(m, "prepare"):
                m.prepare(max_positions)

    def cache_need(self):
        needs = []
        for m in (self.left, self.right):
            need = m.cache_need()
            needs.extend(need if isinstance(need, tuple) else [need])
        return tuple(n for n in needs if n.kind != "none")

    def _forward_joined(self, x, step, cache, stream):
        left, right = self.left, self.right
        proj = self.proj(x, out_dtype=torch.float32)
        out = torch.empty((step.n_tokens, left.out_width + right.out_width), dtype=self.runtime.dtype, device=proj.device)
        left.core(proj[:, :left.proj_width], step, cache, out[:, :left.out_width], scale=self.spec.left_scale)
        right.core(proj[:, left.proj_width:], step, cache, out[:, left.out_width:], scale=self.spec.right_scale)
        return self.o.into_stream(out, stream, torch.float32, handoff=getattr(step, "handoff", None) if stream is not None else None)

    def forward(self, x, step, cache, as_pair=False, stream=None):
        """`as_pair`: the caller's next kernel takes the weighted sum itself; it gets a WeightedPair."""
        if self.spec.joined:
            return self._forward_joined(x, step, cache, stream)
        a = self.left.forward(x, step, cache)
        b = self.right.forward(x, step, cache)
        if a.dtype != torch.float32 or b.dtype != torch.float32:
            raise ValueError("mixers that run side by side hand their outputs over in float32")
        if as_pair:
            return WeightedPair(a, self.spec.left_scale, b, self.spec.right_scale)
        out = torch.empty_like(a)
        K.weighted_sum(a, self.spec.left_scale, b, self.spec.right_scale, out)
        return out
