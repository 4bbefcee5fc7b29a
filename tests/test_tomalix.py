"""The Tomalix decoder without a GPU: its configuration, its plan and stored names, what its runs keep in the cache,
and the plain implementation's mechanisms against closed forms."""
import copy
import math

import numpy as np
import pytest

from plain import tomalix_plain as P
from tomalix_tiny import CONFIGS, TOM_A, make_folder, random_tokens


def test_configuration_round_trip_and_errors():
    from burn_lm_b200.config import ConfigError, TomalixConfig
    for cfg in CONFIGS.values():
        typed = TomalixConfig.from_dict(cfg)
        assert TomalixConfig.from_dict(typed.to_dict()) == typed and typed.to_dict() == cfg
        assert len(typed.layers) == len(cfg["layers"])
    for path, value, key in ((("layers", 0, "type"), "conv", "layers[0].type"),
                             (("layers", 0, "mixer", "rot", "dims"), 7, "layers[0].mixer.rot.dims"),
                             (("layers", 0, "mixer", "rot", "dims"), 18, "layers[0].mixer.rot.dims"),
                             (("layers", 0, "mixer", "kv_heads"), 3, "layers[0].mixer.heads"),
                             (("layers", 0, "mixer", "diff"), None, "layers[0].mixer.diff"),
                             (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0, "layers[0].mixer.rot.scaling.factor"),
                             (("layers", 2, "mixer", "rot", "scaling", "slow"), None, "layers[2].mixer.rot.scaling.slow"),
                             (("layers", 2, "mixer", "rot", "base"), 1.0, "layers[2].mixer.rot.base"),
                             (("layers", 1, "mixer", "left", "mask", "size"), 0, "layers[1].mixer.left.mask.size"),
                             (("layers", 1, "mixer", "left", "rot", "scaling"), {"factor": 2.0}, "layers[1].mixer.left.rot.scaling"),
                             (("layers", 1, "mixer", "right", "state"), 0, "layers[1].mixer.right.state"),
                             (("layers", 1, "mixer", "right", "dt_rank"), None, "layers[1].mixer.right.dt_rank"),
                             (("layers", 1, "mixer", "left_scale"), None, "layers[1].mixer.left_scale"),
                             (("layers", 0, "mlp", "router", "top"), 7, "layers[0].mlp.router.top"),
                             (("layers", 0, "mlp", "kind"), "glu", "layers[0].mlp.kind"),
                             (("layers", 1, "mlp", "ff"), None, "layers[1].mlp.ff"),
                             (("loop", "stop"), 9, "loop"), (("norm", "eps"), "x", "norm.eps"), (("width",), 0, "width")):
        bad = copy.deepcopy(TOM_A)
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=key.replace("[", r"\[").replace("]", r"\]").replace(".", r"\.")):
            TomalixConfig.from_dict(bad)


def test_the_plan_names_the_stored_tensors():
    from burn_lm_b200.model import plan_of, tensor_specs_of
    arch, typed, plan = plan_of(TOM_A)
    assert arch.name == "Tomalix" and plan.head.tensors == {"weight": "head"} and plan.embedding.tensors == {"table": "embed"}
    assert [lp.block for lp in plan.layers] == ["prenorm"] * 6
    assert [(e.layer, e.before) for e in plan.schedule] == [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (4, None), (5, None)]
    assert [lp.part("mixer").kind for lp in plan.layers] == ["normed_attention", "parallel_mixers", "normed_attention", "parallel_mixers"] + ["normed_attention"] * 2
    names = {s.name: tuple(s.shape) for s in tensor_specs_of(TOM_A)}
    assert names["embed"] == (272, 96) and names["head"] == (272, 96) and names["final.norm"] == (96,) and names["loop.step"] == (2, 96)
    assert names["l0.mix.q"] == (4 * 2 * 16, 96) and names["l0.mix.k"] == (2 * 2 * 16, 96) and names["l0.mix.v"] == (64, 96) and names["l0.mix.o"] == (96, 128)
    assert all(names[f"l0.mix.{n}"] == (16,) for n in ("lq1", "lk1", "lq2", "lk2")) and names["l0.norm1"] == (96,)
    assert names["l1.mix.left.q"] == (96, 96) and names["l1.mix.left.v"] == (80, 96) and names["l1.mix.left.g"] == (160, 96) and names["l1.mix.left.o"] == (96, 160)
    assert names["l1.mix.right.in"] == (256, 96) and names["l1.mix.right.conv"] == (128, 4) and names["l1.mix.right.conv.b"] == (128,)
    assert names["l1.mix.right.x"] == (40, 128) and names["l1.mix.right.dt"] == (128, 8) and names["l1.mix.right.dt.b"] == (128,)
    assert names["l1.mix.right.A_log"] == (128, 16) and names["l1.mix.right.D"] == (128,) and names["l1.mix.right.o"] == (96, 128)
    assert names["l0.mlp.router"] == (6, 96) and names["l0.mlp.router.b"] == (6,) and names["l0.mlp.e5.up"] == (48, 96) and names["l0.mlp.e5.down"] == (96, 48)
    assert names["l1.mlp.up"] == (160, 96) and names["l1.mlp.down"] == (96, 160)
    assert "l2.norm2" not in names and "l2.mlp.up" not in names and "l0.mlp.e6.up" not in names and "l2.mix.g" not in names


def test_heads_the_dense_decoder_has_kernels_for_run_its_mixer():
    from burn_lm_b200.model import plan_of
    _, _, plan = plan_of(CONFIGS["tom_d"])
    kinds = [lp.part("mixer").kind for lp in plan.layers]
    assert kinds == ["normed_attention", "attention", "parallel_mixers", "attention", "parallel_mixers", "normed_attention"]


def test_what_the_runs_keep():
    import torch
    from burn_lm_b200.model import Model, plan_of
    from burn_lm_b200.parts.base import Runtime
    _, _, plan = plan_of(TOM_A)
    model = Model(plan, Runtime(torch.float32, "cpu"), TOM_A)
    needs = model.cache_needs()
    assert len(needs) == 9                                             # every pass over the looped layers keeps a line of its own
    assert (needs[0].kind, needs[0].n_kv_heads, needs[0].head_dim, needs[0].value_dim, needs[0].window, needs[0].chunk) == ("kv", 2, 32, 32, None, None)
    kv, state = needs[1]
    assert (kv.kind, kv.n_kv_heads, kv.head_dim, kv.value_dim, kv.chunk) == ("kv", 2, 24, 40, 80)
    assert state.kind == "state" and state.state_shape == (2, 3 * 128 + 128 * 16)
    assert sorted(set(model.kernel_modules()) - {"gemm", "gemm_tc"}) == ["attention_sink", "elementwise", "moe", "recurrent", "stream_ops"]


def test_a_chunked_line_gives_back_the_pages_of_the_chunks_before():
    from burn_lm_b200.parts.base import CacheNeed
    need = CacheNeed("kv", n_kv_heads=1, head_dim=8, chunk=100)
    assert [need.first_needed(n) for n in (0, 1, 99, 100, 101, 199, 250)] == [0, 0, 0, 100, 100, 100, 200]
    assert CacheNeed("kv", window=10).first_needed(25) == 16 and CacheNeed("kv").first_needed(25) == 0


def test_folders_hold_what_the_plain_implementation_reads(tmp_path):
    folder = make_folder(tmp_path, "tom_c")
    cfg, tensors = P.read_model_folder(folder)
    after = []
    logits = P.forward(cfg, tensors, random_tokens(0, 40, cfg["vocab"]), after)
    assert logits.shape == (40, cfg["vocab"]) and len(after) == 12 and np.isfinite(logits).all()
    # causal: a later token changes nothing before it
    again = P.forward(cfg, tensors, random_tokens(0, 40, cfg["vocab"])[:35] + [3, 1, 4, 1, 5])
    assert np.abs(again[:35] - logits[:35]).max() < 1e-12 and np.abs(again[35:] - logits[35:]).max() > 1e-3
    # the package's random-weights mode writes the same names and shapes
    from burn_lm_b200 import write_random_model
    other = write_random_model(str(tmp_path / "r"), cfg, seed=1, dtype="float32")
    _, drawn = P.read_model_folder(other)
    assert set(drawn) == set(tensors) and all(drawn[k].shape == tensors[k].shape for k in tensors)
    assert np.isfinite(P.forward(cfg, drawn, [1, 2, 3])).all()


# rotations: the product's constants against the plain ones, and both against what they should do ------------------------
@pytest.mark.parametrize("dims,base,scaling", [(56, 2e6, (5.0, 1024, 24.0, 1.0)), (24, 500000.0, (8.0, 256, 16.0, 1.0)), (16, 1000.0, (3.0, 64, 8.0, 2.0)),
                                               (64, 1e4, (40.0, 4096, 32.0, 1.0)), (2, 1e4, (2.0, 100, 4.0, 1.0)), (128, 5e5, (1.0, 512, 1.0, 1.0))])
def test_frequencies_scaled_by_lanes(dims, base, scaling):
    from burn_lm_b200.parts.position import RotarySpec, YarnScaling, rotary_inverse_frequencies, rotary_multiplier
    spec = RotarySpec(dims, base, rotary_dim=dims, scaling=YarnScaling(*scaling))
    want, mult = P.yarn_frequencies({"dims": dims, "base": base, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))})
    assert np.allclose(rotary_inverse_frequencies(spec), want, rtol=1e-12) and abs(rotary_multiplier(spec) - mult) < 1e-12
    plain = P.plain_frequencies({"dims": dims, "base": base})
    # between the plain frequency and the divided one; lanes that turn often keep theirs, lanes that turn seldom have it divided
    assert (want <= plain * (1 + 1e-12)).all() and (want >= plain / scaling[0] * (1 - 1e-12)).all()
    turns = scaling[1] * plain / (2 * math.pi)
    if dims >= 48 and scaling[0] > 1:
        assert np.allclose(want[turns > 2 * scaling[2]], plain[turns > 2 * scaling[2]])
        assert np.allclose(want[turns < scaling[3] / 2], plain[turns < scaling[3] / 2] / scaling[0])


def test_divided_frequencies():
    from burn_lm_b200.parts.position import LinearScaling, RotarySpec, rotary_inverse_frequencies, rotary_multiplier
    spec = RotarySpec(16, 100.0, rotary_dim=8, scaling=LinearScaling(2.5))
    assert np.allclose(rotary_inverse_frequencies(spec), [100.0 ** (-2.0 * i / 8) / 2.5 for i in range(4)]) and rotary_multiplier(spec) == 1.0


def test_plain_rotation_depends_on_the_distance_only():
    rng = np.random.default_rng(1)
    q, k, freq = rng.normal(size=(1, 1, 12)), rng.normal(size=(1, 1, 12)), P.plain_frequencies({"dims": 8, "base": 100.0})
    turn = lambda x, p: P.rotate_halves(x, np.array([float(p)]), 8, freq)
    dots = [float((turn(q, i) * turn(k, j)).sum()) for i, j in ((5, 2), (13, 10), (103, 100))]
    assert np.allclose(dots, dots[0])
    assert np.array_equal(turn(q, 9)[..., 8:], q[..., 8:]) and np.array_equal(turn(q, 0), q)
    one = np.zeros((1, 8))
    one[0, 0] = 1.0
    turned = P.rotate_halves(one, np.array([1.0]), 8, freq)
    assert np.allclose(turned[0, [0, 4]], [np.cos(1.0), np.sin(1.0)]) and np.allclose(turned[0, [1, 2, 3, 5, 6, 7]], 0)


# mechanisms against closed forms ----------------------------------------------------------------------------------------
def test_plain_norm_has_the_epsilon_inside_the_root_and_its_weight_around_zero():
    assert np.allclose(P.rms(np.full((1, 4), 1e-3), 1e-2), 1e-3 / np.sqrt(1e-6 + 1e-2))
    assert np.allclose(P.rms_norm(np.array([[3.0, -4.0]]), np.array([1.0, -0.5]), 0.0), [[3.0 / np.sqrt(12.5) * 2, -4.0 / np.sqrt(12.5) * 0.5]])


def test_plain_chunks_start_at_multiples():
    seen = P.chunked(7, 3)
    assert [list(np.nonzero(r)[0]) for r in seen] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]


def test_plain_difference_of_equal_maps_is_a_normed_map():
    rng = np.random.default_rng(2)
    a = rng.normal(size=(3, 2, 8))
    assert np.allclose(P.difference_of_maps(a, a, 0.25, 0.4, 0.0), P.rms(a, 0.0) * 0.6)
    w = {n: np.full(4, v) for n, v in (("lq1", 0.5), ("lk1", 0.2), ("lq2", 0.1), ("lk2", -0.3))}
    assert abs(P.difference_weight(w, 0.4) - (math.exp(0.4) - math.exp(-0.12) + 0.4)) < 1e-12


def test_plain_scan_with_a_constant_input_is_a_geometric_sum():
    T, dt, a = 9, 0.3, -1.7
    x, B, C = np.full((T, 1), 2.0), np.full((T, 1), 0.5), np.full((T, 1), 3.0)
    y = P.selective_scan(x, np.full((T, 1), dt), np.array([[a]]), B, C, np.array([0.25]))
    want = [3.0 * 0.5 * 2.0 * dt * sum(math.exp(a * dt * k) for k in range(t + 1)) + 0.25 * 2.0 for t in range(T)]
    assert np.allclose(y[:, 0], want)


def test_plain_convolution_has_the_current_token_last():
    y = P.convolution(np.array([[1.0], [10.0], [100.0]]), np.array([[0.5, 2.0]]), np.array([7.0]))
    assert np.allclose(y[:, 0], [9.0, 27.5, 212.0])


def test_plain_router_weighs_the_chosen_logits_only():
    h, router = np.array([[1.0, 0.0]]), np.array([[1.0, 0.0], [3.0, 0.0], [0.0, 5.0], [2.0, 0.0]])
    ids, w = P.route(h, router, np.array([0.0, 0.0, 2.5, -5.0]), 2)
    assert ids.tolist() == [[1, 2]] and np.allclose(w, [[1 / (1 + math.exp(-0.5)), 1 / (1 + math.exp(0.5))]])


def test_plain_passes_add_their_vector_and_all_but_the_first_the_embedding():
    x, x0, steps = np.ones((2, 3)), np.full((2, 3), 10.0), np.array([[1.0] * 3, [2.0] * 3])
    assert np.allclose(P.before_pass(x, x0, steps, 0), 2.0) and np.allclose(P.before_pass(x, x0, steps, 1), 13.0)
    order = P.run_order({"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 2}})
    assert order == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None), (4, None)]
