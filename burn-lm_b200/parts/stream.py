"""Rewrites of the residual stream that stand between runs of layers (family "stream").

A stream part takes the stream, what the run before left to be added to it, and the embedding's output of the step, and
returns the stream that the next run reads: forward(resid, delta, embedded, step) -> resid.  A plan lists its stream
parts and names, per run of its schedule, the one that stands in front of it.

Kind "concat_projection": x <- W [x; x0] with W [width, 2 width] (the stream's columns first) and x0 the embedding's
output: a loop over some layers feeds the input in again at the start of every pass.

Kind "pass_entry": x <- x + steps[t], and (where `rejoin` says so) from the second pass on x <- x + x0 + steps[t]: pass t of a loop
has a stored vector of its own, and the embedding's output joins again.

A stream part that only adds to the stream what a norm's kernel can add (`passes_pending`) runs nothing: join(delta) returns what
is then pending.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import kernels as K
from ..registry import register_part
from ..weights.loader import TensorSpec
from .base import Part
from .linear import Linear
from .norm import PendingSum


@dataclass(frozen=True)
class ConcatProjectionSpec:
    hidden_size: int


@register_part("stream", "concat_projection")
class ConcatProjection(Part):
    family = "stream"
    graph_safe = True
    needs_embedding = True        # the model keeps the embedding's output of the step for this part
    roles = ("weight",)
    kernel_modules = ("stream_ops",)

    def tensor_specs(self):
        d = self.spec.hidden_size
        return [TensorSpec(self.tensor_names["weight"], (d, 2 * d))]

    def bind(self, loaded):
        self.linear = Linear(loaded[self.tensor_names["weight"]])

    def forward(self, resid, delta, embedded, step):
        n, d = resid.shape
        both = torch.empty((n, 2 * d), dtype=self.linear.weight.dtype, device=resid.device)
        K.pack_cols(resid, delta, both, 0)          # the pending output joins the stream on the way (fp32)
        K.pack_cols(embedded, None, both, d)
        return self.linear(both, out_dtype=torch.float32)


@dataclass(frozen=True)
class PassEntrySpec:
    hidden_size: int
    passes: int                   # rows of the stored table
    number: int                   # the pass this part stands in front of, from 0
    rejoin: bool = True           # the embedding's output joins again from the second pass on


@register_part("stream", "pass_entry")
class PassEntry(Part):
    family = "stream"
    graph_safe = True
    roles = ("steps",)
    kernel_modules = ("stream_ops",)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.needs_embedding = spec.rejoin and spec.number > 0
        self.passes_pending = not spec.rejoin

    def tensor_specs(self):
        return [TensorSpec(self.tensor_names["steps"], (self.spec.passes, self.spec.hidden_size), init="normal:0.1")]

    def bind(self, loaded):
        self.step = loaded[self.tensor_names["steps"]][self.spec.number].to(torch.float32).contiguous()

    def forward(self, resid, delta, embedded, step):
        if isinstance(delta, PendingSum):
            delta.add(resid)
            delta = None
        K.pass_entry(resid, delta, embedded if self.needs_embedding else None, self.step)
        return resid

    def join(self, delta):
        """What is pending for the norm that reads the stream next: what was, and the pass's vector."""
        return PendingSum.of(delta).and_(PendingSum(biases=(self.step,)))
