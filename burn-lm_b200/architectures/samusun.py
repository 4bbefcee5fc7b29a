"""The Samusun decoder as a plan of parts: the registry entry "Samusun".

A scaled token embedding; layers whose mixer and feed-forward read one norm's output side by side; a mixer per layer that is
attention over a sliding window in which the keys are their own values (biased projections, no rotation, a bias by distance per
head, queries scaled by a number that grows with their position), or retention (a matrix of decayed key-value products per head,
rotated queries and keys, a norm and a gate on every head's output); a dense gated feed-forward, a mixture of gated experts
whose weights are softmax scores over all experts as they are, or none; a last norm, the output projection, scaled and capped
logits.  A span of the layers may run several times in a row with the same weights, every pass with a cache line or state of
its own; before every pass its own vector joins the stream.  Every layer brings its own sizes.  Stored names: 'embed',
'loop.step', 'l<i>.norm1', 'l<i>.mix.*', 'l<i>.mlp.*', 'final.norm', 'head'.
"""
from __future__ import annotations

from ..config.samusun import DenseConfig, SamusunConfig
from ..parts.embedding import CappedHeadSpec, ScaledEmbeddingSpec
from ..parts.feed_forward import SwiGLUSpec
from ..parts.moe import RoutedMoESpec
from ..parts.norm import RMSNormSpec
from ..parts.normed_attention import NormedAttentionSpec
from ..parts.retention import RetentionSpec
from ..parts.stream import PassEntrySpec
from ..plan import LayerPlan, ModelPlan, NamedPart, PartPlan, ScheduleEntry
from ..registry import Architecture, register_architecture
from .tomalix import run_order

MAX_POSITIONS = 1 << 20     # positions enter by distance, by decay and by angle; the cache sets the real limit


def head_slopes(n_heads: int) -> tuple:
    """What a position of distance takes off a head's scores: 2^(-8 (h + 1) / heads)."""
    return tuple(2.0 ** (-8.0 * (h + 1) / n_heads) for h in range(n_heads))


def _mixer(width: int, eps: float, kind: str, m, a: str) -> PartPlan:
    if kind == "attention":
        tensors = {"q": a + "q", "k": a + "k", "o": a + "o", "q_bias": a + "q.b", "k_bias": a + "k.b", "o_bias": a + "o.b"}
        return PartPlan("normed_attention", NormedAttentionSpec(
            hidden_size=width, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.dim, scale=m.scale, eps=eps,
            qk_norm=False, value_norm=False, head_temperature=False, sink=False, window=m.window, values_are_keys=True,
            projection_bias=True, output_bias=True, slopes=head_slopes(m.heads),
            query_temperature=(m.q_temp.coef, m.q_temp.every) if m.q_temp is not None else None), tensors)
    return PartPlan("retention", RetentionSpec(
        hidden_size=width, n_heads=m.heads, key_dim=m.dim, value_dim=m.vdim, decay=m.decay, eps=eps,
        rotary_dims=m.rot.dims if m.rot is not None else 0, rotary_base=m.rot.base if m.rot is not None else 1.0),
        {r: a + r for r in ("q", "k", "v", "g", "o")})


def _feed_forward(width: int, f, a: str) -> PartPlan:
    if isinstance(f, DenseConfig):
        return PartPlan("swiglu", SwiGLUSpec(width, f.ff), {r: a + r for r in ("gate", "up", "down")})
    return PartPlan("routed_moe", RoutedMoESpec(width, f.experts, f.top, f.ff, scores="softmax", renormalise=False),
                    {"router": a + "router", "gate": a + "e{}.gate", "up": a + "e{}.up", "down": a + "e{}.down"})


def samusun_plan(cfg: SamusunConfig) -> ModelPlan:
    width, eps = cfg.width, cfg.eps
    norm = lambda name: PartPlan("rmsnorm", RMSNormSpec(width, eps), {"weight": name})
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = [NamedPart("norm", "norm", norm(p + "norm1")),
                 NamedPart("mixer", "mixer", _mixer(width, eps, layer.type, layer.mixer, p + "mix."))]
        if layer.mlp is not None:
            parts.append(NamedPart("feed_forward", "feed_forward", _feed_forward(width, layer.mlp, p + "mlp.")))
        layers.append(LayerPlan("parallel", tuple(parts)))
    passes = cfg.loop.times if cfg.loop is not None and cfg.loop.stop > cfg.loop.start else 0
    return ModelPlan(
        architecture=cfg.architecture,
        vocab_size=cfg.vocab,
        hidden_size=width,
        embedding=PartPlan("scaled_table", ScaledEmbeddingSpec(cfg.vocab, width, cfg.embedding_scale), {"table": "embed"}),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i, before=t) for i, t in run_order(len(layers), cfg.loop)),
        final_norm=norm("final.norm"),
        head=PartPlan("capped_linear", CappedHeadSpec(cfg.vocab, width, cfg.logit_softcap, cfg.logit_scale), {"weight": "head"}),
        max_positions=MAX_POSITIONS,
        stream_parts=tuple(PartPlan("pass_entry", PassEntrySpec(width, passes, t, rejoin=False), {"steps": "loop.step"}) for t in range(passes)),
        ignorable_tensors=(r"loop\.step",) if passes == 0 else (),
    )


SAMUSUN = register_architecture(Architecture(
    name="Samusun", config_class=SamusunConfig, plan=samusun_plan, aliases=("samusun",),
    description="parallel layers: attention over a window whose keys are its values, with a bias by distance, or retention; dense "
                "or routed gated feed-forward; a looped span of layers; scaled, capped logits"))
