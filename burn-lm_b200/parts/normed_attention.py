"""Grouped-query attention with options on its queries, keys, values, scores, mask and output: normed heads, a turn of some
lanes, a number per head on the scores, capped scores, a sink in the softmax, a window or chunks, two maps a head whose
difference is taken, a gate on every lane, values that are the keys, a bias by distance, queries scaled by their position.

q = Wq h, k = Wk h, v = Wv h, without biases or with (`projection_bias`).  With `qk_norm` every head of q and of k is divided by its root mean square and
multiplied by a weight of the head's size that all heads share; the first `rotary_dims` lanes of every q and k head then turn
by position * f_i, f_i = base^(-2i / rotary_dims) or scaled as `rotary_scaling` says (parts.position), lanes (2i, 2i + 1)
together (`rotary_halves`: lanes (i, i + rotary_dims / 2)); with `value_norm` every head of v is divided by its root mean
square and cached so.  Query head h reads key/value head h // (heads / kv heads); keys have `head_dim` lanes, values `value_dim`.
s = scale * t_h * q.k (`head_temperature`: t a stored number per query head), then s <- cap tanh(s / cap) (`softcap`);
position i sees j <= i, or only 0 <= i - j < window, or only the j of its own chunk of the sequence; p_j = exp(s_j) / (sink +
sum exp(s_j)) with `sink` one more entry of score 0 that carries no value.  With `output_gate` every lane of the heads' outputs
is multiplied by sigmoid(Wg h).  The heads' outputs are concatenated and projected by Wo (plus a bias with `output_bias`).

`values_are_keys`: one projection (with its bias) serves as key and as value, Wv does not exist and the cache keeps one line.
`query_temperature` (coef, every): q is multiplied by 1 + coef ln(floor((position + 1) / every) + 1).  `slopes` (a number per
query head): slope_h * (i - j) is taken off a score, after the cap.

`diff` makes it differential attention: q has two queries and k two keys a head, [head][map][head_dim], each pair an attention
of its own over the head's one value; with lambda = exp(lq1.lk1) - exp(lq2.lk2) + diff the head's output is a_1 - lambda a_2,
divided by its root mean square and multiplied by 1 - diff.

Norms, rotation, scores, cap, softmax and the difference are fp32 in both dtypes.  The projections run as one product with a
fused [q; k; v; g] weight whose result stays in fp32; the attention kernels are the windowed family's
(`kernels.attention_sink`), which take all of this as options.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from .. import kernels as K
from ..registry import register_part
from ..weights.loader import TensorSpec
from .attention import streaming_splits
from .base import CacheNeed, Part
from .linear import Linear
from .norm import PendingSum
from .position import RotarySpec, rotary_inverse_frequencies, rotary_multiplier

BLOCKS_PER_SM = 4          # blocks of the single-token kernels a step should offer every multiprocessor
TABLE_BYTES = 64 << 20     # a layer's table of cosines and sines at most
STREAM_PAGES = 20          # pages a block of the streaming kernel walks before a sequence's keys are cut
NO_WINDOW = 1 << 30        # what the kernels take for "every earlier key"


@dataclass(frozen=True)
class NormedAttentionSpec:
    hidden_size: int
    n_heads: int
    n_kv_heads: int
    head_dim: int                     # lanes of a head's query and key
    value_dim: int                    # lanes of a head's value
    scale: float
    eps: float                        # of the norms over heads
    rotary_dims: int = 0              # how many of a head's first lanes turn
    rotary_base: float = 10000.0
    rotary_halves: bool = False       # lanes (i, i + rotary_dims / 2) turn together instead of (2i, 2i + 1)
    qk_norm: bool = True              # RMS norm with a shared weight over every head of q and of k
    value_norm: bool = True           # every head of v divided by its root mean square
    head_temperature: bool = True     # a stored number per query head multiplies its scores
    softcap: Optional[float] = None   # s <- cap tanh(s / cap)
    sink: bool = True                 # one more entry of score 0 in the softmax's denominator
    window: Optional[int] = None      # None: every earlier key
    chunk: Optional[int] = None       # instead of a window: the keys of the position's own chunk of this many
    rotary_scaling: object = None     # parts.position.LinearScaling, YarnScaling or Llama3Scaling
    output_gate: bool = False         # sigmoid(Wg h) on every lane of the heads' outputs
    diff: Optional[float] = None      # two maps a head, and this constant in the weight of the second
    values_are_keys: bool = False
    projection_bias: bool = False     # biases on q, k and v
    output_bias: bool = False
    query_temperature: Optional[tuple] = None    # (coef, every)
    slopes: Optional[tuple] = None    # a number per query head: what a position of distance takes off its scores


@register_part("mixer", "normed_attention")
class NormedAttention(Part):
    family = "mixer"
    graph_safe = True
    roles = ("q", "k", "v", "o", "g", "q_bias", "k_bias", "v_bias", "o_bias", "q_norm", "k_norm", "temperature", "lq1", "lk1", "lq2", "lk2")
    kernel_modules = ("elementwise", "attention_sink")

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        if spec.n_heads % spec.n_kv_heads:
            raise ValueError(f"{spec.n_heads} heads do not divide into {spec.n_kv_heads} kv heads")
        if spec.value_dim > 512:
            raise ValueError(f"value_dim {spec.value_dim}: the attention kernels take values of up to 512 lanes")
        if spec.rotary_dims % 2 or spec.rotary_dims > spec.head_dim:
            raise ValueError(f"{spec.rotary_dims} turning lanes of {spec.head_dim}: an even number, at most all of them")
        if spec.window is not None and spec.window < 1:
            raise ValueError(f"a window of {spec.window}")
        if spec.chunk is not None and (spec.chunk < 1 or spec.window is not None):
            raise ValueError(f"chunks of {spec.chunk} with a window of {spec.window}: one of the two, at least 1")
        if spec.values_are_keys and (spec.value_dim != spec.head_dim or spec.value_norm or spec.diff is not None):
            raise ValueError(f"values that are the keys have their {spec.head_dim} lanes, no norm of their own and one map a head")
        if spec.slopes is not None and (len(spec.slopes) != spec.n_heads or spec.diff is not None):
            raise ValueError(f"{len(spec.slopes)} slopes for {spec.n_heads} heads of one map")
        if spec.query_temperature is not None and (spec.query_temperature[1] < 1 or spec.query_temperature[1] != int(spec.query_temperature[1])):
            raise ValueError(f"a query temperature that steps every {spec.query_temperature[1]} positions")
        self.maps = 1 if spec.diff is None else 2
        self.q_cols, self.k_cols = self.maps * spec.n_heads * spec.head_dim, self.maps * spec.n_kv_heads * spec.head_dim
        self.v_cols = 0 if spec.values_are_keys else spec.n_kv_heads * spec.value_dim
        self.bias_roles = [r for r in ("q", "k", "v") if spec.projection_bias and not (r == "v" and spec.values_are_keys)]
        self.out_width = spec.n_heads * spec.value_dim
        self.proj_width = self.q_cols + self.k_cols + self.v_cols + (self.out_width if spec.output_gate else 0)

    def tensor_specs(self):
        s, t = self.spec, self.tensor_names
        specs = [TensorSpec(t["q"], (self.q_cols, s.hidden_size)),
                 TensorSpec(t["k"], (self.k_cols, s.hidden_size)),
                 TensorSpec(t["o"], (s.hidden_size, self.out_width))]
        if not s.values_are_keys:
            specs.insert(2, TensorSpec(t["v"], (self.v_cols, s.hidden_size)))
        cols = {"q": self.q_cols, "k": self.k_cols, "v": self.v_cols}
        specs += [TensorSpec(t[r + "_bias"], (cols[r],), init="normal:0.1") for r in self.bias_roles]
        if s.output_bias:
            specs.append(TensorSpec(t["o_bias"], (s.hidden_size,), init="normal:0.1"))
        if s.output_gate:
            specs.append(TensorSpec(t["g"], (self.out_width, s.hidden_size)))
        if s.diff is not None:
            specs += [TensorSpec(t[r], (s.head_dim,), init="normal:0.1") for r in ("lq1", "lk1", "lq2", "lk2")]
        if s.qk_norm:
            specs += [TensorSpec(t["q_norm"], (s.head_dim,), init="one_plus_normal:0.1"),
                      TensorSpec(t["k_norm"], (s.head_dim,), init="one_plus_normal:0.1")]
        if s.head_temperature:
            specs.append(TensorSpec(t["temperature"], (s.n_heads,), init="one_plus_normal:0.1"))
        return specs

    def bind(self, loaded):
        s, t = self.spec, self.tensor_names
        ws = [loaded[t[r]] for r in ("q", "k", "v", "g") if not (r == "v" and s.values_are_keys) and (r != "g" or s.output_gate)]
        if len({w.dtype for w in ws}) != 1:
            raise ValueError(f"the projections of {t['q']} and its neighbours are stored in different dtypes")
        self.proj = Linear(torch.cat(ws, dim=0).contiguous())
        self.o = Linear(loaded[t["o"]])
        f32 = lambda x: x.to(torch.float32).contiguous()
        self.q_weight = f32(loaded[t["q_norm"]]) if s.qk_norm else None
        self.k_weight = f32(loaded[t["k_norm"]]) if s.qk_norm else None
        self.temperature = f32(loaded[t["temperature"]]) if s.head_temperature else None
        self.bias = torch.cat([f32(loaded[t[r + "_bias"]]) for r in self.bias_roles]).contiguous() if self.bias_roles else None
        self.o_bias = f32(loaded[t["o_bias"]]) if s.output_bias else None
        self.slopes = torch.tensor(s.slopes, dtype=torch.float64).to(torch.float32).to(self.o.weight.device) if s.slopes is not None else None
        self.freq, self.turn_scale, self.table = None, 1.0, None
        if s.rotary_dims:
            rot = RotarySpec(s.head_dim, s.rotary_base, rotary_dim=s.rotary_dims, scaling=s.rotary_scaling)
            self.freq = torch.tensor(rotary_inverse_frequencies(rot), dtype=torch.float64).to(self.o.weight.device)
            self.turn_scale = rotary_multiplier(rot)
        self.streams = (s.values_are_keys and self.o.weight.is_cuda and not (s.sink or s.softcap or s.head_temperature or s.output_gate or s.chunk)
                        and K.attention_sink_streams(self.runtime.dtype, s.head_dim, s.n_heads, s.n_kv_heads))
        self.difference = (0.0, 1.0, 0.0)
        if s.diff is not None:
            lq1, lk1, lq2, lk2 = (loaded[t[r]].to(torch.float64) for r in ("lq1", "lk1", "lq2", "lk2"))
            lam = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + s.diff
            self.difference = (lam, 1.0 - s.diff, s.eps)

    def prepare(self, max_positions: int) -> None:
        """Cosines and sines of the positions the cache can hold, worked out once (beyond TABLE_BYTES: by the kernel, a token
        at a time)."""
        if self.freq is not None and self.freq.is_cuda and 8 * self.freq.numel() * max_positions <= TABLE_BYTES \
                and (self.table is None or self.table.shape[0] < max_positions):
            self.table = K.rope_table(self.freq, max_positions, self.turn_scale)

    def cache_need(self) -> CacheNeed:
        s = self.spec
        return CacheNeed("kv", n_kv_heads=s.n_kv_heads, head_dim=self.maps * s.head_dim, window=s.window,
                         value_dim=0 if s.values_are_keys else s.value_dim, chunk=s.chunk)

    def _splits(self, step) -> int:
        """Over how many blocks the single-token kernels cut a row's keys: a few tokens with many keys leave most of the
        multiprocessors idle otherwise."""
        s = self.spec
        if K.attention_sink_prompt_takes(self.runtime.dtype, s.head_dim, s.value_dim, step.max_q_len, self.maps * s.n_heads):
            return 1
        seen = min(step.max_kv_len, s.window or s.chunk or step.max_kv_len)
        if self.streams and step.max_q_len == 1 and step.n_tokens == step.n_seqs:
            return streaming_splits(step.n_seqs, s.n_kv_heads, (seen + 2 * K.PAGE - 2) // K.PAGE, STREAM_PAGES, self.runtime.device)
        blocks = step.n_tokens * self.maps * s.n_kv_heads
        if self.maps == 2 and K.attention_sink_pairs(self.runtime.dtype, s.head_dim, s.value_dim, 2 * s.n_heads, 2 * s.n_kv_heads, 2):
            blocks //= 2                                     # both maps of a head share a block
        want = BLOCKS_PER_SM * K.sm_count(self.runtime.device)
        if K.attention_sink_decode_takes(self.runtime.dtype, s.head_dim, s.value_dim, s.n_heads, s.n_kv_heads):
            pages = seen // K.PAGE + 1                       # that kernel cuts by pages, and its blocks hold several
            want //= 2
            return max(1, min((want + blocks - 1) // blocks, pages // 4, 32))
        return max(1, min((want + blocks - 1) // blocks, seen // 128, 32))

    takes_pending_norm = True
    adds_to_stream = True

    def forward(self, x, step, cache, stream=None):
        rt = self.runtime
        proj = self.proj(x, out_dtype=torch.float32)            # [N, q | k | v (| g)] in fp32
        out = torch.empty((step.n_tokens, self.out_width), dtype=rt.dtype, device=proj.device)
        self.core(proj, step, cache, out)
        y = self.o.into_stream(out, stream, torch.float32, handoff=getattr(step, "handoff", None) if stream is not None else None, bias=self.o_bias)
        return y if y is None or self.o_bias is None else PendingSum((y,), (self.o_bias,))

    # for a block that runs this part's last product and a feed-forward's as one (parts.block.ParallelBlock)
    def output_bias(self):
        return self.o_bias

    def before_output(self, x, step, cache, out):
        """What the output product reads, into `out` [N, out_width] in the compute dtype (it may be a column range)."""
        self.core(self.proj(x, out_dtype=torch.float32), step, cache, out)

    # what two mixers that run side by side with one product in front and one behind ask for (parts.parallel_mixers)
    def input_weight(self):
        return self.proj.weight

    def output_weight(self):
        return self.o.weight

    def core(self, proj, step, cache, out, scale=1.0):
        """What lies between the projections: proj float32 [N, proj_width], out [N, out_width] in the compute dtype, times
        `scale`; either may be a column range of a wider tensor."""
        s, rt, maps = self.spec, self.runtime, self.maps
        if not cache.writes:
            raise ValueError("this mixer appends to a cache line of its own; it cannot read another run's")
        n, heads, kv_heads = step.n_tokens, self.maps * s.n_heads, self.maps * s.n_kv_heads
        q = torch.empty((n, self.q_cols), dtype=rt.dtype, device=proj.device)
        K.head_norm_rope_append(proj, step, cache.pool, cache.block_table, q, heads, kv_heads, s.head_dim, s.value_dim,
                                q_weight=self.q_weight, k_weight=self.k_weight, eps=s.eps, value_norm=s.value_norm, freq=self.freq,
                                rotary_dims=s.rotary_dims, halves=s.rotary_halves, turn_scale=self.turn_scale, maps=maps, table=self.table,
                                bias=self.bias, temperature=s.query_temperature, shared=s.values_are_keys)
        n_splits = self._splits(step)
        prompt = K.attention_sink_prompt_takes(rt.dtype, s.head_dim, s.value_dim, step.max_q_len, heads)
        inside = maps == 2 and not prompt and K.attention_sink_pairs(rt.dtype, s.head_dim, s.value_dim, heads, kv_heads, maps)
        floats = K.attention_sink_scratch_floats(n, heads, s.value_dim, n_splits, maps, inside)
        scratch = None
        if floats and step.max_q_len == 1:
            scratch = step.workspace.scratch("attention_sink", floats)
        elif floats:                            # (a prompt's shares: captured prompt steps share their memory)
            scratch = torch.empty(floats, dtype=torch.float32, device=proj.device)
        gate = proj[:, self.proj_width - self.out_width:] if s.output_gate else None
        K.attention_sink(q, step, cache.pool, cache.block_table, out, heads, kv_heads, s.head_dim, s.value_dim, s.scale,
                         s.window or NO_WINDOW, 0, sink=s.sink, gate=gate, gate_stride=proj.stride(0), max_q_len=step.max_q_len,
                         n_splits=n_splits, scratch=scratch, head_scale=self.temperature, softcap=s.softcap or 0.0, chunk=s.chunk or 0,
                         gate_lanes=s.value_dim if s.output_gate else 0, out_scale=scale, maps=maps, difference=self.difference,
                         slope=self.slopes, shared=s.values_are_keys)
