"""The Samusun decoder in the engine against the plain implementation (tests/plain/samusun_plain.py): every
mechanism alone (its part and kernels on a cache of the test's own), then whole models through the step function, the
cache, the scheduler and generation."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from plain import samusun_plain as P
from samusun_tiny import CONFIGS, dense, experts, make_folder, model, random_tokens, retain, row_error, values, window

pytestmark = pytest.mark.gpu

FP32_TOL = 1e-4
BF16_TOL = 6e-2
PAGE = 64
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dev(x, dtype=torch.float32):
    return torch.tensor(np.asarray(x), dtype=dtype, device="cuda")


def ints(x):
    return torch.tensor(list(x), dtype=torch.int32, device="cuda")


def bf(x):
    """What a bfloat16 tensor holds of x, in float64: weights and inputs that both dtypes read alike."""
    return torch.tensor(np.asarray(x), dtype=torch.float32).to(torch.bfloat16).to(torch.float64).numpy()


class Scratch:
    def scratch(self, name, n):
        return torch.empty(max(n, 1), dtype=torch.float32, device="cuda")


def step_of(portions, slots, starts):
    """A step that brings portions[s] tokens of the sequence in slots[s], which has starts[s] tokens already."""
    seq_of, pos, cu = [], [], [0]
    for s, (k, st) in enumerate(zip(portions, starts)):
        seq_of += [s] * k
        pos += list(range(st, st + k))
        cu.append(cu[-1] + k)
    return SimpleNamespace(token_seq=ints(seq_of), token_pos=ints(pos), slot_of_seq=ints(slots), cu_seqlens=ints(cu),
                           start_pos=ints(starts), n_tokens=len(seq_of), n_seqs=len(slots), max_q_len=max(portions),
                           max_kv_len=max(s + k for s, k in zip(starts, portions)), workspace=Scratch(), memo={}, host={}, handoff=None)


def engine_for(folder, dtype, max_tokens=4096, **kw):
    from burn_lm_b200 import Engine
    return Engine.from_folder(folder, dtype=dtype, max_tokens=max_tokens, **kw)


def rows_ok(err, dtype, tol):
    """float32: nineteen rows in twenty within tol and none beyond 10 tol.  bfloat16: half of the rows within tol / 2 and nine
    in ten within tol (rounding may decide a close call between two experts, which moves a row by far more than rounding)."""
    err = np.atleast_1d(np.asarray(err))
    if dtype == "float32":
        ok = np.quantile(err, 0.95) < tol and err.max() < 10 * tol
    else:
        ok = np.median(err) < tol / 2 and np.quantile(err, 0.9) < tol
    if not ok:
        print(f"{dtype}: median {np.median(err):.3g}, nine in ten {np.quantile(err, 0.9):.3g}, largest {err.max():.3g} of {len(err)} rows")
    return ok


def folder_for(tmp_path, name, dtype, **kw):
    """Lively weights for the sharp comparison in float32, calm ones for bfloat16 (see rows_ok)."""
    return make_folder(tmp_path, name, lively=dtype == "float32", **kw)


# ---------------------------------------------------------------------------------------------------------
# a mixer alone: the part with weights of the test's own, on pages and states of the test's own
# ---------------------------------------------------------------------------------------------------------
def mixer_plan(entry, width, eps=1e-5):
    from burn_lm_b200.model import plan_of
    return plan_of(model(16, width, [entry], eps=eps))[2].layers[0].part("mixer")


def built(plan, dtype, device="cuda"):
    from burn_lm_b200.parts.base import Runtime
    from burn_lm_b200.registry import part_class
    return part_class("mixer", plan.kind)(plan.spec, plan.tensors, Runtime(DTYPES[dtype], torch.device(device)))


def bound(plan, weights, dtype):
    part = built(plan, dtype)
    part.bind({s.name: dev(weights[s.name], DTYPES[dtype]) for s in part.tensor_specs()})
    return part


def mixer_weights(plan, rng):
    return {s.name: bf(values(rng, s.name, tuple(s.shape))) for s in built(plan, "float32", "cpu").tensor_specs()}


def short(weights, prefix="l0.mix."):
    return {k[len(prefix):]: v for k, v in weights.items()}


def joined(y, x):
    """What a part returned for input x, in float64: a tensor, or outputs and biases still to be added."""
    from burn_lm_b200.parts.norm import PendingSum
    p = PendingSum.of(y)
    total = sum(o.double() for o in p.outputs) + sum(b.double() for b in p.biases)
    return total.cpu().numpy()


class OwnCache:
    """Pages of one run, handed out in a shuffled order, with rubbish (NaN) wherever nothing was written; a state block that
    holds rubbish as well (a sequence's start must not read it)."""

    def __init__(self, part, dtype, n_slots=4, pages_each=24, seed=0):
        need = part.cache_need()
        if need.kind == "state":
            self.state = torch.full((n_slots, *need.state_shape), float("nan"), dtype=torch.float32, device="cuda")
        else:
            n_pages = n_slots * pages_each + 3
            self.pool = torch.full((n_pages, need.n_kv_heads * PAGE * (need.head_dim + need.value_dim)), float("nan"), dtype=DTYPES[dtype], device="cuda")
            order = np.random.default_rng(seed).permutation(n_pages)[:n_slots * pages_each]
            self.block_table = ints(order).view(n_slots, pages_each).contiguous()
        self.state_offset, self.writes = 0, True


def run_mixer(part, cache, hs, slots, schedule, dtype):
    """Feeds sequences hs[s] ([T_s, D] arrays) side by side, schedule = list of per-sequence portions; returns every
    sequence's output rows [T_s, D]."""
    if hasattr(part, "prepare"):
        part.prepare(100)                       # (a table for some of the positions, the rest are worked out)
    at, outs = [0] * len(hs), [[] for _ in hs]
    for portion in schedule:
        live = [s for s, k in enumerate(portion) if k > 0]
        st = step_of([portion[s] for s in live], [slots[s] for s in live], [at[s] for s in live])
        x = dev(np.concatenate([hs[s][at[s]:at[s] + portion[s]] for s in live]), DTYPES[dtype])
        y = joined(part.forward(x, st, cache), x)
        row = 0
        for s in live:
            outs[s].append(y[row:row + portion[s]])
            row += portion[s]
            at[s] += portion[s]
    assert at == [len(h) for h in hs]
    return [np.concatenate(o) for o in outs]


SCHEDULES = {
    "whole": lambda a, b: [(a, b)],
    "portions": lambda a, b: [(1, 1), (2, 1), (1, 2), (61, 3), (2, 0), (a - 100, b - 7), (33, 0)],
    "twos": lambda a, b: [(a - 40, b)] + [(2, 0)] * 20,
    "single tokens": lambda a, b: [(a - 30, b - 3)] + [(1, 1)] * 3 + [(1, 0)] * 27,
}


def check_mixer(entry, plain, width, lengths, slots, schedule, dtype, tol, seed):
    rng = np.random.default_rng(seed)
    plan = mixer_plan(entry, width)
    w = mixer_weights(plan, rng)
    hs = [bf(rng.normal(size=(n, width))) for n in lengths]
    part = bound(plan, w, dtype)
    got = run_mixer(part, OwnCache(part, dtype, seed=seed), hs, slots, schedule, dtype)
    for g, h in zip(got, hs):
        want = plain(h, short(w), entry["mixer"])
        assert np.abs(g - want).max() < tol * np.abs(want).max()


ATTENTION_SHAPES = {      # heads, kv heads, lanes, window
    "small heads": (4, 2, 16, 50),
    "one head, a window of one": (1, 1, 32, 1),
    "a window of two": (2, 2, 24, 2),
    "no multiples of eight": (5, 1, 12, 33),
    "heads of 64, a window of a page": (8, 2, 64, 64),
    "heads of 64, every earlier token": (4, 4, 64, None),
    "heads of 128, a window beyond two pages": (4, 1, 128, 150),
    "heads of 72": (2, 2, 72, 65),
    "heads of 120": (3, 1, 120, 1000),
    "heads of 200": (2, 1, 200, 127),
    "seventeen heads a group": (17, 1, 16, 90),
    "heads of 300": (2, 2, 300, 40),
}


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("shape", sorted(ATTENTION_SHAPES))
@pytest.mark.parametrize("schedule", sorted(SCHEDULES))
def test_attention_whose_keys_are_its_values_alone(shape, schedule, dtype, tol):
    H, G, d, size = ATTENTION_SHAPES[shape]
    entry = window(H, G, d, size, None, q_temp=(0.4, 16))
    check_mixer(entry, P.attention, 48, (200, 9), [2, 0], SCHEDULES[schedule](200, 9), dtype, tol, H + d)


RETENTION_SHAPES = {      # heads, key lanes, value lanes, turning lanes
    "small heads": (4, 16, 32, 16),
    "one head, one value lane": (1, 32, 1, 0),
    "no multiples of eight": (5, 12, 20, 6),
    "odd values": (3, 18, 7, 10),
    "heads of 64": (4, 64, 64, 64),
    "heads of 128, some lanes turning": (2, 128, 128, 64),
    "values of 200, keys of 256": (1, 256, 200, 256),
    "values of 512": (1, 64, 512, 32),
    "keys of 300": (1, 300, 40, 20),
    "values of 600": (1, 24, 600, 8),
}


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("shape", sorted(RETENTION_SHAPES))
@pytest.mark.parametrize("schedule", sorted(SCHEDULES))
def test_retention_alone(shape, schedule, dtype, tol):
    H, d, e, rot = RETENTION_SHAPES[shape]
    entry = retain(H, d, e, None, rot_dims=rot, base=300.0)
    check_mixer(entry, lambda h, w, m: P.retention(h, w, m, 1e-5), 48, (200, 9), [1, 3], SCHEDULES[schedule](200, 9), dtype, tol, H + d + e)


@pytest.mark.parametrize("d", [64, 72, 88, 104, 128])
@pytest.mark.parametrize("size", [100, 64, 257, None])
def test_long_portions_of_large_heads(d, size):
    """Portions of several tiles of query rows, beside one another, that start inside windows and pages (the tcgen05 kernel);
    the rows of a page no key has been written to hold NaN.  A steep head beside flat ones: eight slopes from 1/2 to 1/256."""
    rng = np.random.default_rng(d)
    entry = window(8, 2, d, size, None, q_temp=(0.2, 50))
    plan = mixer_plan(entry, 40)
    w = mixer_weights(plan, rng)
    hs = [bf(rng.normal(size=(n, 40))) for n in (500, 300)]
    part = bound(plan, w, "bfloat16")
    for schedule in ([(500, 300)], [(290, 1), (110, 199), (100, 100)], [(64, 64), (65, 127), (371, 109)]):
        got = run_mixer(part, OwnCache(part, "bfloat16"), hs, [2, 0], schedule, "bfloat16")
        for g, h in zip(got, hs):
            want = P.attention(h, short(w), entry["mixer"])
            assert np.abs(g - want).max() < 3e-2 * np.abs(want).max(), schedule


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 2e-2)])
@pytest.mark.parametrize("shape", ["small heads", "no multiples of eight", "heads of 64", "values of 512", "keys of 300"])
def test_retention_over_several_sequences_through_used_states(shape, dtype, tol):
    H, d, e, rot = RETENTION_SHAPES[shape]
    rng = np.random.default_rng(d + e)
    entry = retain(H, d, e, None, rot_dims=rot)
    plan = mixer_plan(entry, 40)
    w = mixer_weights(plan, rng)
    part = bound(plan, w, dtype)
    cache = OwnCache(part, dtype, n_slots=6)
    for lengths, schedule in (((170, 33, 1, 5, 2), [(135, 33, 1, 4, 1), (33, 0, 0, 0, 0), (1, 0, 0, 1, 1), (1, 0, 0, 0, 0)]),
                              ((9, 130, 64, 2, 65), [(8, 130, 32, 1, 64), (1, 0, 32, 1, 1)])):
        hs = [bf(rng.normal(size=(n, 40))) for n in lengths]
        got = run_mixer(part, cache, hs, [4, 0, 2, 5, 1], schedule, dtype)
        for g, h in zip(got, hs):
            want = P.retention(h, short(w), entry["mixer"], 1e-5)
            err = np.abs(g - want).max(axis=1) / np.abs(want).max()
            # (bfloat16: a head whose sum cancels, at a sequence's first tokens mostly, is normed all the same, rounding and all)
            assert np.median(err) < tol and err.max() < (8 * tol if dtype == "bfloat16" else tol)


def retention_rows(q, k, v, g):
    return np.concatenate([x.reshape(len(x), -1) for x in (q, k, v, g)], axis=1)


@pytest.mark.parametrize("dtype,tol", [("float32", 2e-5), ("bfloat16", 1e-2)])
def test_single_token_steps_leave_the_state_they_read_alone(dtype, tol):
    """A step of one token may be run twice (a warm-up in front of a captured graph): it gives the same rows both times."""
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(4)
    n, H, d, e = 3, 2, 20, 24
    state0 = rng.normal(size=(n, 2, H * d * e))
    q, k, v, g = (rng.normal(size=(n, H, x)) for x in (d, d, e, e))
    decay = np.array([0.75, 0.99])
    want_s = decay[:, None, None] * state0[:, 1].reshape(n, H, d, e) + (0.3 * k)[..., None] * v[:, :, None]
    o = np.einsum("nhde,nhd->nhe", want_s, q)
    want = P.rms(o, 1e-5) * P.silu(g)
    st = step_of([1] * n, list(range(n)), [3] * n)
    state, out = dev(state0), torch.empty((n, H * e), dtype=DTYPES[dtype], device="cuda")
    powers = K.retention_powers(decay).cuda()
    for _ in range(2):
        K.retention(dev(retention_rows(q, k, v, g)), st, state, 0, H, d, e, 0.3, powers, 1e-5, out)
        assert np.abs(out.double().cpu().numpy() - want.reshape(n, -1)).max() < tol * np.abs(want).max()
        assert torch.equal(state[:, 1], dev(state0)[:, 1])          # position 3 reads copy 1 and writes copy 0
        assert np.abs(state[:, 0].double().cpu().numpy() - want_s.reshape(n, -1)).max() < 1e-5 * np.abs(want_s).max()


@pytest.mark.parametrize("cuts", [[2100], [1, 63, 65, 700, 1271], [2097, 1, 1, 1], [64] * 32 + [52], [2] * 30 + [2040]])
def test_a_state_remembers_far_back(cuts):
    """A head that hardly decays and one that does not: a key at the first token is still there two thousand tokens later; the
    queries in between read nothing, the values in between are small."""
    from burn_lm_b200 import kernels as K
    T, H, d, e = sum(cuts), 2, 16, 16
    rng = np.random.default_rng(6)
    q, k, v, g = np.zeros((T, H, d)), np.zeros((T, H, d)), np.zeros((T, H, e)), np.full((T, H, e), 3.0)
    u, val = bf(rng.normal(size=(H, d))), bf(rng.normal(size=(H, e)))
    k[0], v[0], q[-1] = u, val, u
    for t in range(1, T):                                    # other keys lie across the first one
        z = rng.normal(size=(H, d))
        k[t] = bf(z - (z * u).sum(-1, keepdims=True) / (u * u).sum(-1, keepdims=True) * u)
        v[t] = 0.01 * rng.normal(size=(H, e))
    decay = np.array([0.9995, 1.0])
    o, _ = P.retain(q, k, v, decay)
    want = (P.rms(o[-1], 1e-5) * P.silu(3.0)).reshape(-1)
    assert np.abs(want - (P.rms(val, 0.0) * P.silu(3.0)).reshape(-1)).max() < 0.2        # the test is sharp: the first value comes back
    rows, powers = dev(retention_rows(q, k, v, g)), K.retention_powers(decay).cuda()
    for dtype, tol in ((torch.float32, 1e-4), (torch.bfloat16, 2e-2)):
        state, at, last = torch.full((1, 2, H * d * e), float("nan"), device="cuda"), 0, None
        for n in cuts:
            st, x = step_of([n], [0], [at]), rows[at:at + n]
            out = torch.zeros((n, H * e), dtype=dtype, device="cuda")
            if dtype == torch.bfloat16:
                K.retention(x, st, state, 0, H, d, e, 1.0, powers, 1e-5, out)
                last = out[-1]
            else:
                K.retention_scan(x, st, state, 0, H, d, e, 1.0, powers, out)
                last = dev((P.rms(out[-1].double().cpu().numpy().reshape(H, e), 1e-5) * P.silu(3.0)).reshape(-1))
            at += n
        assert np.abs(last.double().cpu().numpy() - want).max() < tol * np.abs(want).max()


def test_rows_of_no_sequence_and_empty_sequences():
    """A captured step is padded: rows behind the last sequence change nothing and reach no cache and no state."""
    rng = np.random.default_rng(8)
    for entry in (window(2, 1, 64, 40, None), retain(2, 16, 24, None)):
        plan = mixer_plan(entry, 32)
        part = bound(plan, mixer_weights(plan, rng), "bfloat16")
        for lengths in ([70, 3], [1, 1]):
            h = bf(rng.normal(size=(sum(lengths) + 5, 32)))
            outs = []
            for pad in (0, 5):
                cache = OwnCache(part, "bfloat16")
                st = step_of(lengths + ([0, 0] if pad else []), [0, 1] + ([2, 3] if pad else []), [0] * (4 if pad else 2))
                st.token_seq = torch.cat([st.token_seq, ints([-1] * pad)])
                st.token_pos = torch.cat([st.token_pos, ints([0] * pad)])
                st.n_tokens += pad
                out = torch.full((st.n_tokens, part.out_width), float("nan"), dtype=torch.bfloat16, device="cuda")
                part.before_output(dev(h[:st.n_tokens], torch.bfloat16), st, cache, out)
                outs.append(out)
                kept = cache.state[2:] if hasattr(cache, "state") else cache.pool[cache.block_table[2:].flatten().long()]
                assert torch.isnan(kept.float()).all()
            assert torch.equal(outs[0], outs[1][:sum(lengths)])


# one key made to stand out among hundreds ----------------------------------------------------------------
def planted(n, j, d, size, heads=1):
    """The query reads the first half of the input's lanes and the key the second half, so that the last token's query points
    along the key of token j and along no other token's (its own too); the output is the keys' weighted sum, plus a bias."""
    rng = np.random.default_rng(n + j)
    zero, eye = np.zeros((d, d)), np.eye(d)
    h, u = bf(rng.normal(size=(n, 2 * d))), bf(rng.normal(size=d))
    h[n - 1, :d] = u
    h[j, d:] = u
    w = {"q": np.vstack([np.hstack([eye, zero])] * heads), "q.b": np.zeros(heads * d), "k": np.hstack([zero, eye]), "k.b": bf(0.2 * rng.normal(size=d)),
         "o": bf(rng.normal(size=(2 * d, heads * d)) / np.sqrt(d)), "o.b": bf(rng.normal(size=2 * d))}
    return window(heads, 1, d, size, None, scale=1.5, q_temp=None), w, h


def planted_run(entry, w, h, cuts, dtype, seed):
    part = bound(mixer_plan(entry, h.shape[1]), {"l0.mix." + k: v for k, v in w.items()}, dtype)
    return run_mixer(part, OwnCache(part, dtype, seed=seed), [h], [3], cuts, dtype)[0]


def cuts_of(n, how):
    return {"prompt": [(n,)], "decoded": [(n - 1,), (1,)], "portion": [(n - 2,), (2,)] if n > 2 else [(n,)]}[how]


FAR = [(300, 0), (300, 1), (300, 63), (300, 64), (300, 127), (300, 128), (300, 298), (65, 0), (129, 64), (2, 0)]


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portion"])
@pytest.mark.parametrize("d", [32, 64])
@pytest.mark.parametrize("n,j", FAR)
def test_a_key_far_back_at_page_borders_and_among_the_first_tokens(n, j, d, how, dtype, tol):
    entry, w, h = planted(n, j, d, None)
    want = P.attention(h, w, entry["mixer"])
    key = w["k"] @ h[j] + w["k.b"]
    assert np.abs(want[-1] - (w["o"] @ key + w["o.b"])).max() < 5e-2      # the test is sharp: the last token reads token j and next to nothing else
    got = planted_run(entry, w, h, cuts_of(n, how), dtype, j)
    assert np.abs(got[-1] - want[-1]).max() < tol * np.abs(want[-1]).max() and np.abs(got - want).max() < 3 * tol * np.abs(want).max()


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portion"])
@pytest.mark.parametrize("d", [32, 64])
@pytest.mark.parametrize("n,size,back", [(300, 75, 74), (300, 75, 75), (300, 64, 63), (300, 64, 64), (257, 64, 63), (256, 64, 64), (193, 65, 64), (193, 65, 65),
                                         (300, 2, 1), (300, 2, 2), (301, 300, 299), (301, 300, 300), (150, 200, 149), (130, 129, 128), (130, 129, 129)])
def test_a_key_just_inside_and_just_outside_the_window(n, size, back, d, how, dtype, tol):
    j = n - 1 - back
    entry, w, h = planted(n, j, d, size)
    want = P.attention(h, w, entry["mixer"])
    reads = np.abs(want[-1] - (w["o"] @ (w["k"] @ h[j] + w["k.b"]) + w["o.b"])).max() < 5e-2
    assert reads == (back < size)                             # the test is sharp: all or nothing of token j
    got = planted_run(entry, w, h, cuts_of(n, how), dtype, j)
    assert np.abs(got[-1] - want[-1]).max() < tol * np.abs(want[-1]).max() and np.abs(got - want).max() < 3 * tol * np.abs(want).max()


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portion"])
@pytest.mark.parametrize("d", [32, 64])
@pytest.mark.parametrize("n,j", [(300, 0), (300, 64), (300, 255), (129, 1), (66, 0)])
def test_the_bias_by_distance_decides_between_equal_keys(n, j, d, how, dtype, tol):
    """Two tokens hold the key that the last query points along; every head weighs them by its own slope times the distance
    between them, from all for the nearer to nearly equal."""
    heads = 8
    near = n - 1 - 5
    entry, w, h = planted(n, j, d, None, heads=heads)
    h[near, d:] = h[j, d:]
    h[near, d] += 0.5                                          # not quite equal, so that the weights show
    h = bf(h)
    want = P.attention(h, w, entry["mixer"])
    flat = P.attention(h, w, {**entry["mixer"], "heads": heads})
    assert np.array_equal(want, flat)
    q, keys = h[-1, :d], h[:, d:] + w["k.b"]
    gap = 1.5 * (q @ (keys[near] - keys[j])) + P.slopes(heads) * (near - j)
    assert gap.max() - gap.min() > 10 or near - j < 64         # (the slopes matter)
    got = planted_run(entry, w, h, cuts_of(n, how), dtype, j)
    assert np.abs(got[-1] - want[-1]).max() < tol * np.abs(want[-1]).max() and np.abs(got - want).max() < 3 * tol * np.abs(want).max()


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("every", [1, 10, 64, 100, 1000])
def test_queries_grow_where_the_temperature_steps(every, dtype, tol):
    """With a large coefficient the softmax sharpens from step to step; the steps lie at (p + 1) divisible by `every`."""
    for d in (24, 64):
        entry = window(2, 1, d, 80, None, scale=0.2 if dtype == "float32" else 0.05, q_temp=(1.5, every))
        for schedule in ([(200,)], [(60,), (1,), (1,), (1,), (1,), (1,), (36,)] + [(1,)] * 3 + [(96,)]):
            check_mixer(entry, P.attention, 48, (200,), [1], schedule, dtype, tol, every + d)


def test_a_negative_scale():
    for d in (32, 64, 128):
        entry = window(4, 2, d, 90, None, scale=-0.1)
        for dtype, tol in (("float32", 5e-5), ("bfloat16", 3e-2)):
            check_mixer(entry, P.attention, 64, (150,), [1], [(100,), (30,)] + [(1,)] * 20, dtype, tol, 3)


# the stream, the block, the feed-forwards, the head ------------------------------------------------------------
@pytest.mark.parametrize("width", [72, 96, 2048, 33])
@pytest.mark.parametrize("act", [torch.float32, torch.bfloat16])
def test_pending_sums_join_the_stream_in_front_of_a_norm(width, act):
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(width)
    n = 19
    x, gamma = rng.normal(size=(n, width)), 1.0 + 0.2 * rng.normal(size=width)
    rows = ints([3, 18, 0])
    for kinds, n_biases in (((), 1), ((torch.float32,), 1), ((torch.bfloat16, torch.float32), 0), ((torch.float32, torch.float32), 2)):
        outs = [dev(rng.normal(size=(n, width)), k) for k in kinds]
        biases = [dev(rng.normal(size=width)) for _ in range(n_biases)]
        want = x + sum((o.double().cpu().numpy() for o in outs), 0.0) + sum((b.double().cpu().numpy() for b in biases), 0.0)
        normed = P.rms_norm(want, gamma, 1e-3)
        for gdt in (torch.float32, torch.bfloat16):
            g = dev(gamma, gdt)
            gn = normed / gamma * g.double().cpu().numpy()
            resid, out = dev(x), torch.empty((n, width), dtype=act, device="cuda")
            K.add_rmsnorm_parts(resid, outs, biases, g, 1e-3, out)
            assert np.abs(resid.cpu().numpy() - want).max() < 1e-5
            assert np.abs(out.double().cpu().numpy() - gn).max() < (2e-5 if act == torch.float32 else 2e-2) * np.abs(gn).max()
            resid, out = dev(x), torch.empty((3, width), dtype=act, device="cuda")
            K.add_rmsnorm_parts(resid, outs, biases, g, 1e-3, out, rows)
            assert torch.equal(resid, dev(x))                  # chosen rows leave the stream as it is
            assert np.abs(out.double().cpu().numpy() - gn[[3, 18, 0]]).max() < (2e-5 if act == torch.float32 else 2e-2) * np.abs(gn).max()
        resid = dev(x)
        K.add_rmsnorm_parts(resid, outs, biases, None, 0.0, None)
        assert np.abs(resid.cpu().numpy() - want).max() < 1e-5


@pytest.mark.parametrize("n", [1, 5, 16])
def test_a_bias_joins_the_stream_with_the_skinny_product(n):
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(n)
    m, k = 104, 192
    wt, x, b, s, gamma = bf(rng.normal(size=(m, k)) / np.sqrt(k)), bf(rng.normal(size=(n, k))), rng.normal(size=m), rng.normal(size=(n, m)), rng.normal(size=m)
    want = s + x @ wt.T + b
    wide = dev(np.concatenate([x, x], axis=1), torch.bfloat16)
    for source in (dev(x, torch.bfloat16), wide[:, k:]):                      # rows of their own, or columns of wider ones
        stream = dev(s)
        scaled, squares = torch.empty((n, m), dtype=torch.bfloat16, device="cuda"), torch.empty(((m + 15) // 16, K.SQUARES_ROWS), device="cuda")
        K.gemv(dev(wt, torch.bfloat16), n, x=source, add_into=stream, add_bias=dev(b), hand_over=(dev(gamma), scaled, squares))
        assert np.abs(stream.cpu().numpy() - want).max() < 1e-4
        assert np.abs(squares.sum(0)[:n].cpu().numpy() - (want ** 2).sum(1)).max() < 1e-3 * (want ** 2).sum(1).max()
        assert np.abs(scaled.double().cpu().numpy() - want * gamma).max() < 2e-2 * np.abs(want * gamma).max()


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 2e-2)])
@pytest.mark.parametrize("ff", [None, dense(128), dense(100), experts(4, 2, 40)])
@pytest.mark.parametrize("kind", ["attention", "retention"])
def test_a_layer_adds_both_sublayers_of_one_norm(kind, ff, dtype, tol):
    """The block alone: the sum of both parts joins the stream, with the biases, for few tokens and many, whatever reads the stream
    next; a pending vector joins first."""
    from burn_lm_b200.model import Layer, plan_of
    from burn_lm_b200.parts.base import Runtime
    from burn_lm_b200.parts.norm import PendingSum
    width = 64
    rng = np.random.default_rng(5)
    entry = window(2, 1, 64, 50, ff) if kind == "attention" else retain(2, 32, 64, ff)
    lp = plan_of(model(16, width, [entry]))[2].layers[0]
    layer = Layer(lp, Runtime(DTYPES[dtype], torch.device("cuda")))
    w = {s.name: bf(values(rng, s.name, tuple(s.shape), lively=False)) for p in layer.parts() for s in p.tensor_specs()}
    for p in layer.parts():
        p.bind({s.name: dev(w[s.name], DTYPES[dtype]) for s in p.tensor_specs()})
    layer.block.bound()
    mixer, norm = layer.named["mixer"][1], layer.named["norm"][1]
    loose = 3 if dtype == "bfloat16" and ff is not None and ff["kind"] == "moe" else 1       # (a router of that spread reads rounded rows)
    for n in (1, 7, 16, 70):
        x, vec = rng.normal(size=(n, width)), rng.normal(size=width)
        for pending in (False, True):
            xs = x + vec if pending else x
            h = P.rms_norm(xs, w["l0.norm1"], 1e-5)
            want = xs + P.mixer(h, kind, P.sub(w, "l0.mix."), entry["mixer"], 1e-5)
            if ff is not None:
                want = want + P.feed_forward(h, P.sub(w, "l0.mlp."), ff)
            for next_norm in (None, norm):
                resid, st = dev(x), step_of([n], [1], [0])
                delta = layer.block.forward(resid, PendingSum(biases=(dev(vec),)) if pending else None, st, OwnCache(mixer, dtype), next_norm=next_norm)
                PendingSum.of(delta).add(resid)
                assert np.abs(resid.double().cpu().numpy() - want).max() < loose * tol * np.abs(want).max(), (n, pending)


@pytest.mark.parametrize("cap,scale", [(None, 1.0), (None, 0.3), (9.0, 1.0), (4.0, 2.5), (30.0, -1.5)])
def test_scaled_and_capped_logits(cap, scale):
    from burn_lm_b200.parts.base import Runtime
    from burn_lm_b200.parts.embedding import CappedHead, CappedHeadSpec
    rng = np.random.default_rng(9)
    x, wt = rng.normal(size=(5, 48)), rng.normal(size=(70, 48))
    head = CappedHead(CappedHeadSpec(70, 48, cap, scale), {"weight": "w"}, Runtime(torch.float32, torch.device("cuda")))
    head.bind({"w": dev(wt)})
    want = P.soft_cap(scale * (x @ wt.T), cap)
    assert np.abs(head.forward(dev(x)).cpu().numpy() - want).max() < 1e-5 * np.abs(want).max()


@pytest.mark.parametrize("n_experts,top", [(12, 3), (5, 5), (4, 1), (1, 1), (33, 4)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_routing_by_a_softmax_over_all_experts(n_experts, top, dtype):
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(n_experts + top)
    h, router = bf(rng.normal(size=(45, 40))), bf(3.0 * rng.normal(size=(n_experts, 40)) / np.sqrt(40))
    want_ids, want_w = P.route(h, router, top)
    ids, weights = K.moe_route(dev(h, dtype), dev(router), top, scores=K.SCORES_SOFTMAX, renormalise=False)
    assert np.array_equal(ids.cpu().numpy(), want_ids) and np.allclose(weights.cpu().numpy(), want_w, atol=1e-6)
    if top < n_experts:
        assert (weights.sum(1) < 0.9999).any()                # the weights are the scores, not divided by their sum


@pytest.mark.parametrize("n,width,ff,n_experts,top", [(3, 64, 48, 6, 2), (45, 40, 24, 8, 2), (150, 36, 20, 6, 2), (60, 72, 40, 1, 1), (70, 128, 256, 6, 2),
                                                      (700, 136, 72, 4, 2), (1100, 64, 264, 3, 1), (520, 128, 128, 2, 2), (900, 192, 96, 5, 3)])
def test_gated_experts(n, width, ff, n_experts, top):
    """Every route of the experts' products."""
    from burn_lm_b200.parts.base import Runtime
    from burn_lm_b200.parts.moe import RoutedMoE, RoutedMoESpec
    rng = np.random.default_rng(n)
    h = bf(rng.normal(size=(n, width)))
    w = {"router": bf(6.0 * rng.normal(size=(n_experts, width)) / np.sqrt(width))}
    for e in range(n_experts):
        for r, s in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
            w[f"e{e}.{r}"] = bf(1.5 * rng.normal(size=s) / np.sqrt(s[1]))
    want = P.experts(h, w, experts(n_experts, top, ff))
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 3e-2)):
        part = RoutedMoE(RoutedMoESpec(width, n_experts, top, ff, scores="softmax", renormalise=False),
                         {"router": "router", "gate": "e{}.gate", "up": "e{}.up", "down": "e{}.down"}, Runtime(DTYPES[dtype], torch.device("cuda")))
        part.bind({s.name: dev(w[s.name], DTYPES[dtype]) for s in part.tensor_specs()})
        got = part.forward(dev(h, DTYPES[dtype]), SimpleNamespace(handoff=None)).double().cpu().numpy()
        assert np.abs(got - want).max() < tol * np.abs(want).max()


# ---------------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------------
def _logits(engine, tokens, want, portions=None):
    from burn_lm_b200 import StepEntry
    slot = engine.acquire()
    rows, at = [], 0
    for k in portions or [len(tokens)]:
        w = [p - at for p in want if at <= p < at + k]
        out = engine.step([StepEntry(slot, tokens[at: at + k], w)])
        if w:
            rows.append(out.cpu().numpy().copy())
        at += k
    engine.release(slot)
    return np.concatenate(rows)


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype,tol", [("float32", FP32_TOL), ("bfloat16", BF16_TOL)])
def test_whole_prompts_portions_and_single_tokens(tmp_path, name, dtype, tol):
    folder = folder_for(tmp_path, name, dtype)
    cfg, tensors = P.read_model_folder(folder)
    tokens = random_tokens(1, 250, cfg["vocab"])
    want = P.forward(cfg, tensors, tokens)
    engine = engine_for(folder, dtype)
    every = list(range(len(tokens)))
    assert rows_ok(row_error(_logits(engine, tokens, every), want), dtype, tol)
    for portions in ([64, 64, 122], [1, 2, 61, 1, 1, 2, 2, 17, 63, 100], [200] + [1] * 50, [2] * 125):
        assert rows_ok(row_error(_logits(engine, tokens, every, portions), want), dtype, tol), portions
    # the first tokens alone, one at a time from an empty sequence
    assert rows_ok(row_error(_logits(engine, tokens[:9], list(range(9)), [1] * 9), want[:9]), dtype, tol)
    engine.verify()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_stream_after_every_layer(tmp_path, name):
    from burn_lm_b200 import StepEntry
    folder = make_folder(tmp_path, name)
    cfg, tensors = P.read_model_folder(folder)
    tokens = random_tokens(2, 40, cfg["vocab"])
    after = []
    P.forward(cfg, tensors, tokens, after)
    engine = engine_for(folder, "float32")
    engine.use_graphs = False
    seen, kept = [], []
    for layer in engine.model.layers:
        block = layer.block

        def watched(resid, delta, step, view, next_norm=None, plain=block.forward):
            pending = plain(resid, delta, step, view, next_norm=next_norm)
            seen.append(resid.cpu().numpy() + joined(pending, resid) if pending is not None else resid.cpu().numpy())      # what is pending joins the stream
            return pending

        kept.append((block, block.forward))
        block.forward = watched
    try:
        slot = engine.acquire()
        engine.step([StepEntry(slot, tokens, [0])])
        engine.release(slot)
    finally:
        for block, plain in kept:
            block.forward = plain
    assert len(seen) == len(after)
    for i, (got, want) in enumerate(zip(seen, after)):
        assert np.abs(got[:len(tokens)] - want).max() < 1e-4 * np.abs(want).max(), i


@pytest.mark.parametrize("name", ["sam_a", "sam_c", "sam_d"])
@pytest.mark.parametrize("dtype,tol", [("float32", FP32_TOL), ("bfloat16", BF16_TOL)])
def test_unequal_requests_together_through_used_slots_and_pages(tmp_path, name, dtype, tol):
    from burn_lm_b200 import StepEntry
    folder = folder_for(tmp_path, name, dtype)
    cfg, tensors = P.read_model_folder(folder)
    engine = engine_for(folder, dtype, max_tokens=1024)
    errs = []
    for set_no in range(3):              # the same slots and pages serve three sets of requests
        lengths = [[1, 70, 230], [65, 3, 64, 120], [228, 2]][set_no]
        reqs = [random_tokens(10 * set_no + i, n + 12, cfg["vocab"]) for i, n in enumerate(lengths)]
        want = [P.forward(cfg, tensors, r) for r in reqs]
        slots = [engine.acquire() for _ in reqs]
        out = engine.step([StepEntry(s, r[:n], [0, n - 1]) for s, r, n in zip(slots, reqs, lengths)]).cpu().numpy()
        for i, n in enumerate(lengths):
            errs += [row_error(out[2 * i], want[i][0]), row_error(out[2 * i + 1], want[i][n - 1])]
            assert dtype != "float32" or max(errs[-2:]) < tol, (set_no, i)
        live = list(range(len(reqs)))
        for t in range(12):
            if t == 5:                      # the shortest request ends early
                gone = live.pop(int(np.argmin([lengths[i] for i in live])))
                engine.release(slots[gone])
            out = engine.step([StepEntry(slots[i], [reqs[i][lengths[i] + t]], [0]) for i in live]).cpu().numpy().copy()
            for j, i in enumerate(live):
                errs.append(row_error(out[j], want[i][lengths[i] + t]))
                assert dtype != "float32" or errs[-1] < tol, (set_no, i, t)
        for i in live:
            engine.release(slots[i])
    engine.verify()
    assert rows_ok(errs, dtype, tol)


def test_prompts_beside_decoded_tokens_in_one_step(tmp_path):
    """A step that brings one token of some sequences and portions of others."""
    from burn_lm_b200 import StepEntry
    folder = make_folder(tmp_path, "sam_a")
    cfg, tensors = P.read_model_folder(folder)
    engine = engine_for(folder, "float32", max_tokens=2048)
    reqs = [random_tokens(70 + i, 200, cfg["vocab"]) for i in range(3)]
    want = [P.forward(cfg, tensors, r) for r in reqs]
    slots, at = [engine.acquire() for _ in reqs], [0, 0, 0]
    for portions in ((79, 1, 24), (1, 80, 1), (1, 1, 70), (2, 1, 1), (1, 17, 2), (90, 100, 102)):
        out = engine.step([StepEntry(s, r[a:a + k], list(range(k))) for s, r, a, k in zip(slots, reqs, at, portions)]).cpu().numpy()
        exp = np.concatenate([w[a:a + k] for w, a, k in zip(want, at, portions)])
        assert row_error(out, exp).max() < FP32_TOL, portions
        at = [a + k for a, k in zip(at, portions)]
    for s in slots:
        engine.release(s)


@pytest.mark.parametrize("name", ["sam_a", "sam_c"])
def test_long_decoding_while_the_windows_give_pages_back(tmp_path, name):
    from burn_lm_b200 import StepEntry
    folder = make_folder(tmp_path, name)
    cfg, tensors = P.read_model_folder(folder)
    tokens = random_tokens(5, 400, cfg["vocab"])
    want = P.forward(cfg, tensors, tokens)
    engine = engine_for(folder, "float32", max_tokens=640)       # room for the keys of every position and little else
    slot = engine.acquire()
    engine.step([StepEntry(slot, tokens[:30], [])])
    for p in range(30, len(tokens)):
        row = engine.step([StepEntry(slot, [tokens[p]], [0])]).cpu().numpy()[0]
        assert row_error(row, want[p]) < FP32_TOL, p
    windowed = [g for g in engine.cache._kv_groups if g.need.window]
    assert windowed and all(len(g.live_pages(slot)) <= (g.need.window + PAGE - 1) // PAGE + 1 for g in windowed)
    engine.release(slot)
    engine.verify()


@pytest.mark.parametrize("name", ["sam_a", "sam_b"])
def test_greedy_generation_through_the_entry_point(tmp_path, name):
    import burn_lm_b200 as blm
    folder = make_folder(tmp_path, name)
    cfg, tensors = P.read_model_folder(folder)
    prompts = [random_tokens(20 + i, n, cfg["vocab"]) for i, n in enumerate([5, 70, 17])]
    want = [P.greedy(cfg, tensors, p, 10) for p in prompts]
    lm = blm.load(folder, dtype="float32", max_seq_len=256, max_batch=3)
    assert lm.generate(prompts, sample_len=10, ignore_stop=True).tokens == want
    assert lm.generate(prompts[::-1], sample_len=10, ignore_stop=True).tokens == want[::-1]      # used slots, another order


def test_the_device_side_decode_loop(tmp_path):
    from burn_lm_b200 import StepEntry
    folder = make_folder(tmp_path, "sam_a")
    cfg, tensors = P.read_model_folder(folder)
    prompts = [random_tokens(30 + i, n, cfg["vocab"]) for i, n in enumerate([33, 64])]
    want = [P.greedy(cfg, tensors, p, 12) for p in prompts]
    engine = engine_for(folder, "float32", max_tokens=1024)
    slots = [engine.acquire() for _ in prompts]
    first = engine.step([StepEntry(s, p, [len(p) - 1]) for s, p in zip(slots, prompts)]).argmax(dim=-1).tolist()
    assert first == [w[0] for w in want]
    more = engine.decode_run(slots, first, 8).cpu().numpy()
    assert more.T.tolist() == [w[1:9] for w in want]
    again = engine.decode_run(slots, [w[8] for w in want], 3)       # the captured graph once more, from where it stopped
    assert again.cpu().numpy().T.tolist() == [w[9:] for w in want]


def test_sampling_with_a_temperature_runs_inside_the_captured_step(tmp_path):
    import burn_lm_b200 as blm
    folder = make_folder(tmp_path, "sam_a")
    lm = blm.load(folder, dtype="bfloat16", max_seq_len=256, max_batch=2)
    prompts = [random_tokens(50, 20, 272), random_tokens(51, 66, 272)]
    a = lm.generate(prompts, sample_len=12, temperature=0.8, seed=7, ignore_stop=True).tokens
    b = lm.generate(prompts, sample_len=12, temperature=0.8, seed=7, ignore_stop=True).tokens
    assert a == b and all(len(t) == 12 for t in a)          # the same draws from the same seed, through used slots


def test_the_trace_runner_as_a_child_process(tmp_path):
    cfg = CONFIGS["sam_c"]
    a, b = random_tokens(40, 115, cfg["vocab"]), random_tokens(41, 9, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:110], "want": [0, 109]}, {"id": "b", "tokens": b[:5], "want": [4]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[110]], "want": []}, {"id": "b", "tokens": [b[5]], "want": [0]}], "end": []}]
    steps += [{"step": 2 + t, "entries": [{"id": "a", "tokens": [a[111 + t]], "want": [0]}] + ([{"id": "b", "tokens": [b[6 + t]], "want": [0]}] if t < 3 else []),
               "end": ["b"] if t == 2 else []} for t in range(4)]
    out = tmp_path / "out"
    for dtype, tol in (("float32", FP32_TOL), ("bfloat16", BF16_TOL)):
        folder = folder_for(tmp_path, "sam_c", dtype)
        cfg, tensors = P.read_model_folder(folder)
        proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                               "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
        wa, wb = P.forward(cfg, tensors, a), P.forward(cfg, tensors, b)
        read = lambda n: np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        want = {0: [wa[0], wa[109], wb[4]], 1: [wb[5]]}
        want.update({2 + t: [wa[111 + t]] + ([wb[6 + t]] if t < 3 else []) for t in range(4)})
        errs = [e for n, w in want.items() for e in row_error(read(n), np.stack(w))]
        assert len(errs) == 11 and rows_ok(errs, dtype, tol), errs


def test_the_command_line_on_the_preset(tmp_path):
    program = [sys.executable, os.path.join(ROOT, "bin", "burn-lm")]
    folder = str(tmp_path / "n")
    r = subprocess.run(program + ["random", folder, "--preset", "samusun_tiny", "--seed", "4", "--dtype", "float32"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and f"wrote {folder}" in r.stdout, r.stderr
    cfg, tensors = P.read_model_folder(folder)
    prompt = random_tokens(5, 23, cfg["vocab"])
    want = P.greedy(cfg, tensors, prompt, 12)
    r = subprocess.run(program + ["run", folder, "--dtype", "float32", "--sample-len", "12", "--max-seq-len", "128",
                                  ",".join(map(str, prompt))], capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr
    lines = [ln for ln in r.stdout.splitlines() if ln.strip()]
    assert lines[0].split() == [str(t) for t in want], (lines[0], want)


@pytest.mark.parametrize("kinds", ["windows only", "retention only", "no feed-forward", "experts only, no loop", "the whole model loops", "an empty loop"])
def test_models_of_one_kind_of_layer_and_other_orders(tmp_path, kinds):
    e, d = experts(6, 2, 32), dense(72)
    layers, loop = {
        "windows only": ([window(4, 2, 16, 20, e), window(2, 2, 24, 100, d)], None),
        "retention only": ([retain(2, 16, 24, d), retain(3, 8, 16, None, rot_dims=4)], (1, 2, 3)),
        "no feed-forward": ([retain(2, 24, 16, None), window(3, 3, 8, 64, None), window(1, 1, 64, 65, None)], (0, 2, 2)),
        "experts only, no loop": ([window(2, 2, 16, 64, e), retain(2, 16, 16, e), window(4, 4, 8, 33, e)], None),
        "the whole model loops": ([window(2, 1, 16, 40, d), retain(2, 16, 32, e, rot_dims=4)], (0, 2, 4)),
        "an empty loop": ([window(2, 1, 64, 90, d), retain(1, 64, 64, d)], (1, 1, 3)),
    }[kinds]
    cfg = model(97, 48, layers, loop=loop)
    tokens = random_tokens(7, 190, 97)
    for dtype, tol in (("float32", FP32_TOL), ("bfloat16", BF16_TOL)):
        folder = folder_for(tmp_path, "m", dtype, seed=3, config=cfg)
        pcfg, tensors = P.read_model_folder(folder)
        want = P.forward(pcfg, tensors, tokens)
        engine = engine_for(folder, dtype)
        assert rows_ok(row_error(_logits(engine, tokens, list(range(190)), [170] + [1] * 20), want), dtype, tol)
        assert rows_ok(row_error(_logits(engine, tokens, list(range(190)), [3, 64, 2, 121]), want), dtype, tol)
