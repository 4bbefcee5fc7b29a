"""The Samusun decoder without a GPU: its configuration, its plan and stored names, what its runs keep in the cache,
and the plain implementation's mechanisms against closed forms."""
import copy
import math

import numpy as np
import pytest

from plain import samusun_plain as P
from samusun_tiny import CONFIGS, SAM_A, make_folder, random_tokens


def test_configuration_round_trip_and_errors():
    from burn_lm_b200.config import ConfigError, SamusunConfig
    for cfg in CONFIGS.values():
        typed = SamusunConfig.from_dict(cfg)
        assert SamusunConfig.from_dict(typed.to_dict()) == typed and typed.to_dict() == cfg
        assert len(typed.layers) == len(cfg["layers"])
    for path, value, key in ((("layers", 0, "type"), "conv", "layers[0].type"),
                             (("layers", 0, "mixer", "rot", "dims"), 7, "layers[0].mixer.rot.dims"),
                             (("layers", 0, "mixer", "rot", "dims"), 18, "layers[0].mixer.rot.dims"),
                             (("layers", 0, "mixer", "decay"), [0.5, 0.5], "layers[0].mixer.decay"),
                             (("layers", 0, "mixer", "decay"), [0.5, 0.5, 1.5], "layers[0].mixer.decay"),
                             (("layers", 0, "mixer", "vdim"), 0, "layers[0].mixer.vdim"),
                             (("layers", 1, "mixer", "vdim"), 32, "layers[1].mixer.vdim"),
                             (("layers", 1, "mixer", "kv_heads"), 3, "layers[1].mixer.heads"),
                             (("layers", 1, "mixer", "scale"), None, "layers[1].mixer.scale"),
                             (("layers", 1, "mixer", "mask", "size"), 0, "layers[1].mixer.mask.size"),
                             (("layers", 1, "mixer", "q_temp", "every"), 0, "layers[1].mixer.q_temp.every"),
                             (("layers", 1, "mixer", "q_temp", "coef"), None, "layers[1].mixer.q_temp.coef"),
                             (("layers", 1, "mlp", "router", "top"), 7, "layers[1].mlp.router.top"),
                             (("layers", 0, "mlp", "kind"), "glu", "layers[0].mlp.kind"),
                             (("layers", 0, "mlp", "ff"), None, "layers[0].mlp.ff"),
                             (("loop", "stop"), 9, "loop"), (("norm", "eps"), "x", "norm.eps"), (("width",), 0, "width"),
                             (("embedding", "scale"), "x", "embedding.scale"), (("logit_scale",), "x", "logit_scale")):
        bad = copy.deepcopy(SAM_A)
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=key.replace("[", r"\[").replace("]", r"\]").replace(".", r"\.")):
            SamusunConfig.from_dict(bad)


def test_the_plan_names_the_stored_tensors():
    from burn_lm_b200.model import plan_of, tensor_specs_of
    arch, typed, plan = plan_of(SAM_A)
    assert arch.name == "Samusun" and plan.head.tensors == {"weight": "head"} and plan.embedding.tensors == {"table": "embed"}
    assert [lp.block for lp in plan.layers] == ["parallel"] * 6
    assert [(e.layer, e.before) for e in plan.schedule] == [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (4, None), (5, None)]
    assert [lp.part("mixer").kind for lp in plan.layers] == ["retention", "normed_attention"] * 2 + ["normed_attention", "retention"]
    names = {s.name: tuple(s.shape) for s in tensor_specs_of(SAM_A)}
    assert names["embed"] == (272, 96) and names["head"] == (272, 96) and names["final.norm"] == (96,) and names["loop.step"] == (2, 96)
    assert names["l0.mix.q"] == (48, 96) and names["l0.mix.k"] == (48, 96) and names["l0.mix.v"] == (96, 96) and names["l0.mix.g"] == (96, 96)
    assert names["l0.mix.o"] == (96, 96) and names["l0.norm1"] == (96,) and names["l0.mlp.gate"] == (160, 96) and names["l0.mlp.down"] == (96, 160)
    assert names["l1.mix.q"] == (96, 96) and names["l1.mix.q.b"] == (96,) and names["l1.mix.k"] == (48, 96) and names["l1.mix.k.b"] == (48,)
    assert names["l1.mix.o"] == (96, 96) and names["l1.mix.o.b"] == (96,) and names["l1.mlp.router"] == (6, 96)
    assert names["l1.mlp.e5.gate"] == (48, 96) and names["l1.mlp.e5.down"] == (96, 48)
    for absent in ("l1.mix.v", "l1.mix.v.b", "l0.mix.q.b", "l1.norm2", "l4.mlp.up", "l1.mlp.e6.up", "l1.mlp.router.b"):
        assert absent not in names


def test_what_the_runs_keep():
    import torch
    from burn_lm_b200.model import Model, plan_of
    from burn_lm_b200.parts.base import Runtime
    _, _, plan = plan_of(SAM_A)
    model = Model(plan, Runtime(torch.float32, "cpu"), SAM_A)
    needs = model.cache_needs()
    assert len(needs) == 9                                             # every pass over the looped layers keeps a line of its own
    assert needs[0].kind == "state" and needs[0].state_shape == (2, 3 * 16 * 32)
    assert (needs[1].kind, needs[1].n_kv_heads, needs[1].head_dim, needs[1].value_dim, needs[1].window) == ("kv", 2, 24, 0, 70)
    assert needs[1].first_needed(100) == 31
    assert sorted(set(model.kernel_modules()) - {"gemm", "gemm_tc"}) == ["attention_sink", "elementwise", "moe", "recurrent", "retention", "stream_ops"]


def test_a_line_whose_values_are_its_keys_holds_the_keys_alone():
    import torch
    from burn_lm_b200.cache.cache import _KVGroup
    from burn_lm_b200.parts.base import CacheNeed
    group = _KVGroup(CacheNeed("kv", n_kv_heads=3, head_dim=16, window=70, value_dim=0), [0, 1], 5, 2, 4, torch.bfloat16, "cpu")
    assert tuple(group.pool.shape) == (2, 5, 3 * 64 * 16)
    both = _KVGroup(CacheNeed("kv", n_kv_heads=3, head_dim=16, window=70), [0, 1], 5, 2, 4, torch.bfloat16, "cpu")
    assert both.pool.numel() == 2 * group.pool.numel()


def test_the_products_slopes_and_powers():
    from burn_lm_b200.architectures.samusun import head_slopes
    from burn_lm_b200.kernels import RETENTION_CHUNK, retention_powers
    for n in (1, 2, 3, 5, 8, 12):
        assert np.allclose(head_slopes(n), P.slopes(n), rtol=1e-12)
    assert head_slopes(8)[0] == 0.5 and head_slopes(8)[7] == 2.0 ** -8 and head_slopes(1) == (2.0 ** -8,)
    p = retention_powers([0.5, 1.0, 0.0, 0.999]).numpy()
    assert p.shape == (4, RETENTION_CHUNK + 1) and p[0, 3] == 0.125 and (p[1] == 1.0).all() and p[2].tolist() == [1.0] + [0.0] * RETENTION_CHUNK
    assert abs(p[3, 64] - 0.999 ** 64) < 1e-7


def test_pending_sums():
    import torch
    from burn_lm_b200.parts.norm import PendingSum
    a, b, c = torch.ones(2, 3), torch.ones(2, 3), torch.ones(3)
    assert PendingSum.of(None).simplest() is None and PendingSum.of(a).simplest() is a
    both = PendingSum.of(a).and_(PendingSum((b,), (c,)))
    assert both.simplest() is both and both.fits() and not both.and_(a).fits()
    assert PendingSum.of((a, b)).outputs == (a, b) and PendingSum.of(both) is both


def test_folders_hold_what_the_plain_implementation_reads(tmp_path):
    folder = make_folder(tmp_path, "sam_c")
    cfg, tensors = P.read_model_folder(folder)
    after = []
    logits = P.forward(cfg, tensors, random_tokens(0, 40, cfg["vocab"]), after)
    assert logits.shape == (40, cfg["vocab"]) and len(after) == 15 and np.isfinite(logits).all()
    # causal: a later token changes nothing before it
    again = P.forward(cfg, tensors, random_tokens(0, 40, cfg["vocab"])[:35] + [3, 1, 4, 1, 5])
    assert np.abs(again[:35] - logits[:35]).max() < 1e-12 and np.abs(again[35:] - logits[35:]).max() > 1e-3
    # the package's random-weights mode writes the same names and shapes
    from burn_lm_b200 import write_random_model
    other = write_random_model(str(tmp_path / "r"), cfg, seed=1, dtype="float32")
    _, drawn = P.read_model_folder(other)
    assert set(drawn) == set(tensors) and all(drawn[k].shape == tensors[k].shape for k in tensors)
    assert np.isfinite(P.forward(cfg, drawn, [1, 2, 3])).all()


# mechanisms against closed forms ----------------------------------------------------------------------------------------
def test_plain_temperature_steps_where_the_count_of_tokens_is_a_multiple():
    t = P.query_temperature(range(10), 0.5, 4)
    assert (t[:3] == 1.0).all() and np.allclose(t[3:7], 1.0 + 0.5 * math.log(2.0)) and np.allclose(t[7:], 1.0 + 0.5 * math.log(3.0))


def test_plain_window_and_bias():
    seen = P.sliding_window(5, 2)
    assert [list(np.nonzero(r)[0]) for r in seen] == [[0], [0, 1], [1, 2], [2, 3], [3, 4]]
    s = P.biased_scores(np.zeros((3, 2)), np.ones((3, 2)), 1.0, 0.25)
    assert np.allclose(s, [[0.0, 0.25, 0.5], [-0.25, 0.0, 0.25], [-0.5, -0.25, 0.0]])


def test_plain_attention_reads_its_keys_as_values():
    k = np.array([[[1.0, 2.0]], [[5.0, -1.0]]])
    q = np.array([[[0.0, 0.0]], [[0.0, 0.0]]])
    out = P.shared_attention(q, k, 1.0, P.sliding_window(2, 2))
    near = 1.0 / (1.0 + math.exp(-2.0 ** -8))               # the nearer key by one position's slope
    assert np.allclose(out[0, 0], k[0, 0]) and np.allclose(out[1, 0], near * k[1, 0] + (1 - near) * k[0, 0])


def test_plain_rotation_depends_on_the_distance_only():
    rng = np.random.default_rng(1)
    q, k = rng.normal(size=(1, 1, 12)), rng.normal(size=(1, 1, 12))
    turn = lambda x, p: P.rotate_halves(x, np.array([float(p)]), 8, 100.0)
    dots = [float((turn(q, i) * turn(k, j)).sum()) for i, j in ((5, 2), (13, 10), (103, 100))]
    assert np.allclose(dots, dots[0])
    assert np.array_equal(turn(q, 9)[..., 8:], q[..., 8:]) and np.array_equal(turn(q, 0), q)
    one = np.zeros((1, 8))
    one[0, 0] = 1.0
    turned = P.rotate_halves(one, np.array([1.0]), 8, 100.0)
    assert np.allclose(turned[0, [0, 4]], [np.cos(1.0), np.sin(1.0)]) and np.allclose(turned[0, [1, 2, 3, 5, 6, 7]], 0)


def test_plain_retention_is_a_decayed_sum():
    rng = np.random.default_rng(2)
    q, k, v = rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 4))
    decay = np.array([0.5, 0.9])
    o, S = P.retain(q, k, v, decay)
    for h in range(2):
        want = sum(decay[h] ** (5 - s) * (q[5, h] @ k[s, h]) * v[s, h] for s in range(6))
        assert np.allclose(o[5, h], want)
    first, mid = P.retain(q[:4], k[:4], v[:4], decay)
    rest, last = P.retain(q[4:], k[4:], v[4:], decay, mid)
    assert np.allclose(np.concatenate([first, rest]), o) and np.allclose(last, S)


def test_plain_router_keeps_its_scores_as_they_are():
    h, router = np.array([[1.0, 0.0]]), np.array([[1.0, 0.0], [3.0, 0.0], [0.0, 5.0], [2.0, 0.0]])
    ids, w = P.route(h, router, 2)
    e = np.exp([1.0, 3.0, 0.0, 2.0])
    assert ids.tolist() == [[1, 3]] and np.allclose(w, [[e[1] / e.sum(), e[3] / e.sum()]]) and w.sum() < 0.95


def test_plain_passes_add_their_vector():
    order = P.run_order({"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 2}})
    assert order == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None), (4, None)]
