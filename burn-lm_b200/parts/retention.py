"""The retention mixer: a matrix of decayed key-value products per head, read by the query; nothing is normalised over the keys.

q = Wq h and k = Wk h (heads x key_dim), v = Wv h (heads x value_dim), without biases.  The first `rotary_dims` lanes of every q
and k head turn by position * base^(-2i / rotary_dims), lanes (i, i + rotary_dims / 2) together; then k is multiplied by
key_dim^(-1/2).  Per head, S [key_dim x value_dim] with a decay of its own that no token changes: S <- decay_h S + k v^T,
o = S^T q.  y = Wo (silu(Wg h) * [o_1 / rms(o_1); o_2 / rms(o_2); ...]), the unit norms without a weight.

The four projections run as one product with a fused [q; k; v; g] weight whose result stays in fp32.  S is fp32 and carried per
sequence, two copies by position as the other recurrences'.  In bfloat16, single tokens run one kernel from the projection to the
gated heads, and longer portions run by chunks of tokens on the tensor cores; the 32-bit path (and head sizes beyond those
kernels) walks the tokens in order with its sums in float64.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import kernels as K
from ..registry import register_part
from ..weights.loader import TensorSpec
from .base import CacheNeed, Part
from .linear import Linear

TABLE_BYTES = 64 << 20     # a layer's table of cosines and sines at most


@dataclass(frozen=True)
class RetentionSpec:
    hidden_size: int
    n_heads: int
    key_dim: int
    value_dim: int
    decay: tuple                  # a number per head
    eps: float                    # of the norm over every head's output
    rotary_dims: int = 0
    rotary_base: float = 10000.0


@register_part("mixer", "retention")
class Retention(Part):
    family = "mixer"
    graph_safe = True
    roles = ("q", "k", "v", "g", "o")
    takes_pending_norm = True
    adds_to_stream = True

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        s = spec
        if len(s.decay) != s.n_heads:
            raise ValueError(f"{len(s.decay)} decays for {s.n_heads} heads")
        if s.rotary_dims % 2 or not 0 <= s.rotary_dims <= s.key_dim:
            raise ValueError(f"{s.rotary_dims} turning lanes of {s.key_dim}: an even number, at most all of them")
        if s.key_dim > 512:
            raise ValueError(f"key_dim {s.key_dim}: the retention kernels take keys of up to 512 lanes")
        self.out_width = s.n_heads * s.value_dim
        self.state_floats = s.n_heads * s.key_dim * s.value_dim
        self.kernel_modules = ("elementwise", "retention", "recurrent") if runtime.exact else ("elementwise", "retention")

    def tensor_specs(self):
        s, t = self.spec, self.tensor_names
        kw, d = s.n_heads * s.key_dim, s.hidden_size
        return [TensorSpec(t["q"], (kw, d)), TensorSpec(t["k"], (kw, d)), TensorSpec(t["v"], (self.out_width, d)),
                TensorSpec(t["g"], (self.out_width, d)), TensorSpec(t["o"], (d, self.out_width))]

    def bind(self, loaded):
        s, t = self.spec, self.tensor_names
        ws = [loaded[t[r]] for r in ("q", "k", "v", "g")]
        if len({w.dtype for w in ws}) != 1:
            raise ValueError(f"the projections of {t['q']} and its neighbours are stored in different dtypes")
        self.proj = Linear(torch.cat(ws, dim=0).contiguous())
        self.o = Linear(loaded[t["o"]])
        device = self.o.weight.device
        self.powers = K.retention_powers(s.decay).to(device)
        half = s.rotary_dims // 2
        self.freq = torch.tensor([s.rotary_base ** (-2.0 * i / s.rotary_dims) for i in range(half)], dtype=torch.float64).to(device) if half else None
        self.table = None
        self.unit = torch.ones(s.value_dim, dtype=torch.float32, device=device)

    def prepare(self, max_positions: int) -> None:
        """Cosines and sines of the positions the cache can hold, worked out once (beyond TABLE_BYTES: by the kernels)."""
        if self.freq is not None and self.freq.is_cuda and 8 * self.freq.numel() * max_positions <= TABLE_BYTES \
                and (self.table is None or self.table.shape[0] < max_positions):
            self.table = K.rope_table(self.freq, max_positions)

    def cache_need(self) -> CacheNeed:
        return CacheNeed("state", state_shape=(2, self.state_floats))

    def forward(self, x, step, cache, stream=None):
        rt = self.runtime
        out = torch.empty((step.n_tokens, self.out_width), dtype=rt.dtype, device=self.o.weight.device)
        self.before_output(x, step, cache, out)
        return self.o.into_stream(out, stream, torch.float32, handoff=getattr(step, "handoff", None) if stream is not None else None)

    # for a block that runs this part's last product and a feed-forward's as one (parts.block.ParallelBlock)
    def output_weight(self):
        return self.o.weight

    def output_bias(self):
        return None

    def before_output(self, x, step, cache, out):
        """What the output product reads, into `out` [N, out_width] in the compute dtype (it may be a column range)."""
        s, rt = self.spec, self.runtime
        if not cache.writes:
            raise ValueError("this mixer carries a state of its own; it cannot read another run's")
        proj = self.proj(x, out_dtype=torch.float32)             # [N, q | k | v | g] in fp32
        turn = dict(freq=self.freq, rotary_dims=s.rotary_dims, table=self.table)
        sizes = (s.n_heads, s.key_dim, s.value_dim, s.key_dim ** -0.5, self.powers)
        takes = K.retention_step_takes if step.max_q_len == 1 else K.retention_chunks_take
        if not rt.exact and takes(s.key_dim, s.value_dim):
            K.retention(proj, step, cache.state, cache.state_offset, *sizes, s.eps, out, **turn)
            return
        o = torch.zeros((step.n_tokens, self.out_width), dtype=torch.float32, device=proj.device)     # rows of no sequence stay zero
        K.retention_scan(proj, step, cache.state, cache.state_offset, *sizes, o, **turn)
        K.gated_group_norm(o, proj, 2 * s.n_heads * s.key_dim + self.out_width, self.unit, s.value_dim, K.GATE_SILU_LAST, s.eps, out)
