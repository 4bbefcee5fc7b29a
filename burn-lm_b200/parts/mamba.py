"""The selective scan mixer (Mamba).

One input projection gives [x | z]; x passes a short causal convolution per channel (with a bias) and silu, and is projected
once more to [dt | B | C]: `dt_rank` lanes the step sizes are made from, and what is written and read of `state` states.  Per
channel c: dt_c = softplus(W_dt dt + bias)_c, S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B[n] with A = -exp(A_log),
y_c = sum_n S[c, n] C[n] + D_c x_c; y silu(z) is projected out.  The convolution's last inputs and S (fp32) are what a sequence
carries from token to token.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import kernels as K
from ..registry import register_part
from ..weights.loader import TensorSpec
from .base import CacheNeed, Part
from .linear import Linear

FUSED_STEP_TOKENS = 16     # up to this many tokens the scan's kernel forms the step sizes itself,
FUSED_STEP_RANK = 2048     # from at most so many lanes


@dataclass(frozen=True)
class MambaSpec:
    hidden_size: int
    inner: int                    # channels
    state: int                    # states of a channel
    conv: int                     # taps of the convolution
    dt_rank: int


def f32(t):
    return t.to(torch.float32).contiguous()


@register_part("mixer", "mamba")
class Mamba(Part):
    family = "mixer"
    graph_safe = True
    roles = ("in", "conv", "conv_bias", "x", "dt", "dt_bias", "A_log", "D", "o")
    kernel_modules = ("recurrent",)
    takes_pending_norm = True

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        s = spec
        if s.state > K.SELECTIVE_STATES:
            raise ValueError(f"{s.state} states a channel; the scan takes up to {K.SELECTIVE_STATES}")
        self.low_width = s.dt_rank + 2 * s.state
        self.proj_width, self.out_width = 2 * s.inner, s.inner
        # one copy of what a sequence carries: the convolution's last inputs, then the channels' states
        self.hist_floats = (s.conv - 1) * s.inner
        self.state_floats = self.hist_floats + s.inner * s.state

    def tensor_specs(self):
        s, t = self.spec, self.tensor_names
        return [TensorSpec(t["in"], (2 * s.inner, s.hidden_size)),
                TensorSpec(t["conv"], (s.inner, s.conv), init="normal:0.3"),
                TensorSpec(t["conv_bias"], (s.inner,), init="normal:0.1"),
                TensorSpec(t["x"], (self.low_width, s.inner)),
                TensorSpec(t["dt"], (s.inner, s.dt_rank)),
                TensorSpec(t["dt_bias"], (s.inner,), init="normal:0.5"),
                TensorSpec(t["A_log"], (s.inner, s.state), init="normal:0.5"),
                TensorSpec(t["D"], (s.inner,), init="one_plus_normal:0.1"),
                TensorSpec(t["o"], (s.hidden_size, s.inner))]

    def bind(self, loaded):
        t = self.tensor_names
        self.proj, self.x, self.dt, self.o = (Linear(loaded[t[r]].contiguous()) for r in ("in", "x", "dt", "o"))
        self.taps, self.conv_bias = f32(loaded[t["conv"]]), f32(loaded[t["conv_bias"]])
        self.dt_bias, self.a_log, self.d_skip = f32(loaded[t["dt_bias"]]), f32(loaded[t["A_log"]]), f32(loaded[t["D"]])
        self.rates = K.scan_rates(self.a_log)

    def cache_need(self) -> CacheNeed:
        return CacheNeed("state", state_shape=(2, self.state_floats))

    def forward(self, x, step, cache):
        proj = self.proj(x, out_dtype=torch.float32)                       # [N, x | z] in fp32
        out = torch.empty((step.n_tokens, self.out_width), dtype=self.runtime.dtype, device=proj.device)
        self.core(proj, step, cache, out)
        return self.o(out, out_dtype=torch.float32)

    def input_weight(self):
        return self.proj.weight

    def output_weight(self):
        return self.o.weight

    def core(self, proj, step, cache, out, scale=1.0):
        """What lies between the projections: proj float32 [N, proj_width], out [N, out_width] in the compute dtype, times
        `scale`; either may be a column range of a wider tensor."""
        s, rt = self.spec, self.runtime
        if not cache.writes:
            raise ValueError("this mixer carries a state of its own; it cannot read another run's")
        n = step.n_tokens
        x = torch.empty((n, s.inner), dtype=torch.float32, device=proj.device)
        rounded = torch.empty((n, s.inner), dtype=torch.bfloat16, device=proj.device) if self.x.weight.dtype == torch.bfloat16 else None
        K.causal_conv(proj, 0, s.inner, self.taps, self.conv_bias, x, 0, step, cache.state, cache.state_offset, silu=True, out_bf16=rounded)
        low = self.x(rounded if rounded is not None else x, out_dtype=torch.float32)            # [N, dt | B | C] in fp32
        dt = None
        if n > FUSED_STEP_TOKENS or step.max_q_len > 1 or s.dt_rank > FUSED_STEP_RANK:
            latent = torch.empty((n, s.dt_rank), dtype=self.dt.weight.dtype, device=proj.device)
            K.take_cols(low, 0, latent)
            dt = self.dt(latent, out_dtype=torch.float32)
        K.selective_scan(x, low, s.dt_rank, s.state, self.dt_bias, self.a_log, self.d_skip, proj[:, s.inner: 2 * s.inner], out, step,
                         cache.state, cache.state_offset + self.hist_floats, dt=dt, dt_weight=self.dt.weight if dt is None else None,
                         scale=scale, rates=self.rates)
