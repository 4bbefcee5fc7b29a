"""The Tomalix decoder as a plan of parts: the registry entry "Tomalix".

A token embedding; pre-norm layers whose norm weights are stored around zero; a mixer per layer that is differential
attention (two maps a head over the same values, their weighted difference normed head by head; frequencies divided by a
factor), grouped-query attention with frequencies scaled by lanes (YaRN), or two mixers side by side: attention inside
chunks of the sequence with a gate on every lane, and a selective scan (Mamba); a dense feed-forward without a gate, a
mixture of such experts whose weights are a softmax over the chosen logits, or none; a last norm, the output projection,
and logits squashed by a tanh cap.  A span of the layers may run several times in a row with the same weights, every pass
with a cache line and state of its own; before a pass its own vector, and before every pass but the first the embedding's
output, join the stream (stream part "pass_entry").  Every layer brings its own sizes.  Stored names: 'embed',
'loop.step', 'l<i>.norm1', 'l<i>.norm2', 'l<i>.mix.*', 'l<i>.mlp.*', 'final.norm', 'head'.
"""
from __future__ import annotations

from ..config.tomalix import DenseConfig, LinearScalingConfig, TomalixConfig
from ..parts.attention import TUNED_HEADS, AttentionSpec
from ..parts.embedding import CappedHeadSpec, EmbeddingSpec
from ..parts.feed_forward import MLPSpec
from ..parts.mamba import MambaSpec
from ..parts.moe import RoutedMoESpec
from ..parts.norm import RMSNormSpec
from ..parts.normed_attention import NormedAttentionSpec
from ..parts.parallel_mixers import ParallelMixersSpec
from ..parts.position import LinearScaling, NoPositionSpec, RotarySpec, YarnScaling
from ..parts.stream import PassEntrySpec
from ..plan import LayerPlan, ModelPlan, NamedPart, PartPlan, ScheduleEntry
from ..registry import Architecture, register_architecture

MAX_POSITIONS = 1 << 20     # the rotation takes any position; the cache sets the real limit
ACTIVATION = "relu2"        # of the dense feed-forward and of the experts, fixed by the design


def _scaling(s):
    if s is None:
        return None
    if isinstance(s, LinearScalingConfig):
        return LinearScaling(s.factor)
    return YarnScaling(factor=s.factor, original_max_position=s.original, fast=s.fast, slow=s.slow)


def _attention(width: int, eps: float, m, a: str, gate: bool = False) -> PartPlan:
    tensors = {r: a + r for r in ("q", "k", "v", "o")}
    if m.diff is None and m.chunk is None and not gate and m.dim == m.vdim and m.dim in TUNED_HEADS and m.scale > 0:
        # nothing but full causal attention, at a head size the dense decoder's mixer has kernels for
        position = PartPlan("none", NoPositionSpec())
        if m.rot.dims:
            position = PartPlan("rotary", RotarySpec(m.dim, m.rot.base, rotary_dim=m.rot.dims, scaling=_scaling(m.rot.scaling)))
        return PartPlan("attention", AttentionSpec(width, m.heads, m.kv_heads, m.dim, position, softmax_scale=m.scale), tensors)
    if m.diff is not None:
        tensors.update({r: a + r for r in ("lq1", "lk1", "lq2", "lk2")})
    if gate:
        tensors["g"] = a + "g"
    return PartPlan("normed_attention", NormedAttentionSpec(
        hidden_size=width, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps,
        rotary_dims=m.rot.dims, rotary_base=m.rot.base, rotary_halves=True, rotary_scaling=_scaling(m.rot.scaling), qk_norm=False,
        value_norm=False, head_temperature=False, sink=False, chunk=m.chunk, output_gate=gate, diff=m.diff), tensors)


def _mixer(width: int, eps: float, kind: str, m, p: str) -> PartPlan:
    a = p + "mix."
    if kind != "parallel":
        return _attention(width, eps, m, a)
    s, b = m.right, a + "right."
    right = PartPlan("mamba", MambaSpec(hidden_size=width, inner=s.inner, state=s.state, conv=s.conv, dt_rank=s.dt_rank),
                     {"in": b + "in", "conv": b + "conv", "conv_bias": b + "conv.b", "x": b + "x", "dt": b + "dt", "dt_bias": b + "dt.b",
                      "A_log": b + "A_log", "D": b + "D", "o": b + "o"})
    return PartPlan("parallel_mixers", ParallelMixersSpec(_attention(width, eps, m.left, a + "left.", gate=True), right, m.left_scale,
                                                          m.right_scale, joined=True))


def _feed_forward(width: int, f, p: str) -> PartPlan:
    if isinstance(f, DenseConfig):
        return PartPlan("mlp", MLPSpec(width, f.ff, ACTIVATION), {"up": p + "mlp.up", "down": p + "mlp.down"})
    return PartPlan("routed_moe", RoutedMoESpec(width, f.experts, f.top, f.ff, scores="chosen_softmax", bias=True, renormalise=False,
                                                unit=ACTIVATION),
                    {"router": p + "mlp.router", "bias": p + "mlp.router.b", "up": p + "mlp.e{}.up", "down": p + "mlp.e{}.down"})


def run_order(n_layers: int, loop) -> list:
    """[(layer, number of the pass that starts with this run, or None)]: the looped span `times` times in a row, the rest once."""
    if loop is None:
        return [(i, None) for i in range(n_layers)]
    order = [(i, None) for i in range(loop.start)]
    for t in range(loop.times):
        order += [(i, t if i == loop.start else None) for i in range(loop.start, loop.stop)]
    return order + [(i, None) for i in range(loop.stop, n_layers)]


def tomalix_plan(cfg: TomalixConfig) -> ModelPlan:
    width, eps = cfg.width, cfg.eps
    norm = lambda name: PartPlan("rmsnorm", RMSNormSpec(width, eps, around_zero=True), {"weight": name})
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = [NamedPart("mixer_norm", "norm", norm(p + "norm1")),
                 NamedPart("mixer", "mixer", _mixer(width, eps, layer.type, layer.mixer, p))]
        if layer.mlp is not None:
            parts += [NamedPart("feed_forward_norm", "norm", norm(p + "norm2")),
                      NamedPart("feed_forward", "feed_forward", _feed_forward(width, layer.mlp, p))]
        layers.append(LayerPlan("prenorm", tuple(parts)))
    passes = cfg.loop.times if cfg.loop is not None and cfg.loop.stop > cfg.loop.start else 0
    return ModelPlan(
        architecture=cfg.architecture,
        vocab_size=cfg.vocab,
        hidden_size=width,
        embedding=PartPlan("table", EmbeddingSpec(cfg.vocab, width), {"table": "embed"}),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i, before=t) for i, t in run_order(len(layers), cfg.loop)),
        final_norm=norm("final.norm"),
        head=PartPlan("capped_linear", CappedHeadSpec(cfg.vocab, width, cfg.logit_softcap), {"weight": "head"}),
        max_positions=MAX_POSITIONS,
        stream_parts=tuple(PartPlan("pass_entry", PassEntrySpec(width, passes, t), {"steps": "loop.step"}) for t in range(passes)),
        ignorable_tensors=(r"loop\.step",) if passes == 0 else (),
    )


TOMALIX = register_architecture(Architecture(
    name="Tomalix", config_class=TomalixConfig, plan=tomalix_plan, aliases=("tomalix",),
    description="pre-norm layers: differential attention, attention with scaled frequencies, or attention in chunks beside a "
                "selective scan; dense or routed squared-relu feed-forward; a looped span of layers; capped logits"))
