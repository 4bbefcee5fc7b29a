"""The Tomalix decoder in the engine against the plain implementation (tests/plain/tomalix_plain.py): every
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

from plain import tomalix_plain as P
from tomalix_tiny import CONFIGS, dense, difference, experts, make_folder, model, pair, random_tokens, row_error, scaled, values

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


class OwnCache:
    """Pages of one run, handed out in a shuffled order, with rubbish (NaN) wherever nothing was written; a state block that
    holds rubbish as well (a sequence's start must not read it)."""

    def __init__(self, part, dtype, n_slots=4, pages_each=24, seed=0):
        needs = part.cache_need()
        for need in needs if isinstance(needs, tuple) else (needs,):
            if need.kind == "state":
                self.state = torch.full((n_slots, *need.state_shape), float("nan"), dtype=torch.float32, device="cuda")
                continue
            n_pages = n_slots * pages_each + 3
            dv = need.value_dim or need.head_dim
            shape = (n_pages, 2, need.n_kv_heads, PAGE, dv) if dv == need.head_dim else (n_pages, need.n_kv_heads * PAGE * (need.head_dim + dv))
            self.pool = torch.full(shape, float("nan"), dtype=DTYPES[dtype], device="cuda")
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
        y = part.forward(x, st, cache).float().cpu().numpy()
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


DIFFERENCE_SHAPES = {      # heads, kv heads, dim, vdim, turning lanes
    "small heads": (4, 2, 16, 32, 16),
    "one head, values as wide as the keys": (1, 1, 32, 32, 8),
    "no multiples of eight": (5, 1, 12, 20, 6),
    "heads of 64 and 128": (4, 2, 64, 128, 64),
    "heads of 128 and 256": (2, 1, 128, 256, 0),
    "heads of 72 and 136": (2, 2, 72, 136, 40),
    "heads of 88 and 184": (2, 1, 88, 184, 48),
    "nine heads a group": (9, 1, 16, 48, 16),
    "values of 320": (2, 2, 24, 320, 24),
}


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 6e-2)])
@pytest.mark.parametrize("shape", sorted(DIFFERENCE_SHAPES))
@pytest.mark.parametrize("schedule", sorted(SCHEDULES))
def test_differential_attention_alone(shape, schedule, dtype, tol):
    H, G, dk, dv, rot = DIFFERENCE_SHAPES[shape]
    entry = difference(H, G, dk, dv, None, rot_dims=rot, base=300.0, factor=2.5, diff=0.35)
    check_mixer(entry, lambda h, w, m: P.differential_attention(h, w, m, 1e-5), 48, (200, 9), [2, 0], SCHEDULES[schedule](200, 9), dtype, tol, H + dk)


SCALED_SHAPES = {
    "small heads": (6, 3, 32, 16, 24),
    "one head": (1, 1, 16, 16, 16),
    "no multiples of eight": (5, 1, 12, 20, 6),
    "heads of 64": (8, 2, 64, 64, 64),
    "heads of 128, some lanes turning": (4, 1, 128, 128, 64),
    "heads of 64, none turning": (2, 2, 64, 64, 0),
    "heads of 96, values of 200": (2, 1, 96, 200, 96),
    "seventeen heads a group": (17, 1, 16, 24, 8),
}


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("shape", sorted(SCALED_SHAPES))
@pytest.mark.parametrize("schedule", sorted(SCHEDULES))
def test_attention_with_scaled_frequencies_alone(shape, schedule, dtype, tol):
    H, G, dk, dv, rot = SCALED_SHAPES[shape]
    entry = scaled(H, G, dk, dv, None, rot_dims=rot, base=300.0, scaling=(6.0, 60, 9.0, 1.0))
    check_mixer(entry, lambda h, w, m: P.full_attention(h, w, m, 1e-5), 48, (200, 9), [1, 3], SCHEDULES[schedule](200, 9), dtype, tol, H + dk)


PAIR_SHAPES = {           # heads, kv heads, dim, vdim, chunk, turning lanes, channels, states, taps, rank
    "small": (4, 2, 24, 40, 80, 12, 128, 16, 4, 8),
    "a chunk of one": (1, 1, 32, 32, 1, 32, 64, 1, 1, 1),
    "a chunk of two": (2, 2, 16, 16, 2, 0, 36, 3, 2, 5),
    "no multiples of eight": (5, 1, 12, 20, 33, 6, 44, 5, 5, 3),
    "a chunk of a page": (4, 1, 64, 64, 64, 32, 256, 20, 4, 12),
    "a chunk beyond two pages, values of 184": (4, 2, 88, 184, 150, 32, 96, 8, 3, 6),
    "a chunk beyond the sequence, values of 256": (2, 1, 128, 256, 1000, 128, 100, 40, 4, 24),
    "many states": (2, 2, 16, 16, 100, 8, 32, 128, 8, 12),
}


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("shape", sorted(PAIR_SHAPES))
@pytest.mark.parametrize("schedule", sorted(SCHEDULES))
def test_chunked_attention_beside_a_selective_scan(shape, schedule, dtype, tol):
    H, G, dk, dv, chunk, rot, C, S, K, R = PAIR_SHAPES[shape]
    entry = pair(H, G, dk, dv, chunk, C, S, K, R, None, rot_dims=rot, base=300.0)
    check_mixer(entry, P.parallel_mixers, 48, (200, 9), [3, 1], SCHEDULES[schedule](200, 9), dtype, tol, H + dk + chunk)


@pytest.mark.parametrize("dk,dv", [(64, 64), (64, 128), (72, 136), (128, 128), (80, 168), (128, 256), (104, 64), (128, 200)])
@pytest.mark.parametrize("kind", ["chunks", "maps"])
def test_long_portions_of_large_heads(kind, dk, dv):
    """Portions of several tiles of query rows, beside one another, that start inside chunks and pages (the tcgen05 kernel);
    the rows of a page no key has been written to hold NaN."""
    rng = np.random.default_rng(dk + dv)
    if kind == "maps":
        entry, plain = difference(2, 1, dk, dv, None, rot_dims=32, base=300.0, diff=0.2, scale=0.5 * dk ** -0.5), lambda h, w, m: P.differential_attention(h, w, m, 1e-5)
        plan = mixer_plan(entry, 40)
    else:
        entry, plain = pair(4, 2, dk, dv, 150, 8, 1, 1, 1, None, rot_dims=32, base=300.0), lambda h, w, m: P.chunk_attention(h, w, m["left"])
        plan = mixer_plan(entry, 40).spec.left
    w = mixer_weights(plan, rng)
    hs = [bf(rng.normal(size=(n, 40))) for n in (500, 300)]
    part = bound(plan, w, "bfloat16")
    prefix = "l0.mix." if kind == "maps" else "l0.mix.left."
    for schedule in ([(500, 300)], [(290, 1), (110, 199), (100, 100)], [(64, 64), (65, 127), (371, 109)]):
        got = run_mixer(part, OwnCache(part, "bfloat16"), hs, [2, 0], schedule, "bfloat16")
        for g, h in zip(got, hs):
            want = plain(h, short(w, prefix), entry["mixer"])
            assert np.abs(g - want).max() < 4e-2 * np.abs(want).max(), schedule


@pytest.mark.parametrize("dtype,tol", [("float32", 5e-5), ("bfloat16", 2e-2)])
@pytest.mark.parametrize("shape", sorted(PAIR_SHAPES))
def test_the_scan_alone_over_several_sequences(shape, dtype, tol):
    """The mixer's scan as a part of its own (not joined to another mixer), five sequences, through states used before."""
    C, S, K, R = PAIR_SHAPES[shape][6:]
    rng = np.random.default_rng(C + S)
    plan = mixer_plan(pair(1, 1, 8, 8, 4, C, S, K, R, None), 40).spec.right
    w = mixer_weights(plan, rng)
    part = bound(plan, w, dtype)
    cache = OwnCache(part, dtype, n_slots=6)
    for lengths, schedule in (((70, 33, 1, 5, 2), [(35, 33, 1, 4, 1), (33, 0, 0, 0, 0), (1, 0, 0, 1, 1), (1, 0, 0, 0, 0)]),
                              ((9, 90, 64, 2, 31), [(8, 90, 32, 1, 30), (1, 0, 32, 1, 1)])):
        hs = [bf(rng.normal(size=(n, 40))) for n in lengths]
        got = run_mixer(part, cache, hs, [4, 0, 2, 5, 1], schedule, dtype)
        m = {"inner": C, "state": S, "dt_rank": R}
        for g, h in zip(got, hs):
            want = P.mamba(h, short(w, "l0.mix.right."), m)
            assert np.abs(g - want).max() < tol * np.abs(want).max()


@pytest.mark.parametrize("S,R,C", [(16, 64, 64), (1, 3, 33), (20, 12, 48), (7, 257, 40), (64, 40, 36), (128, 8, 32)])
def test_scan_kernels_agree_on_step_sizes_formed_inside_and_brought(S, R, C):
    """Single tokens: the step sizes from their projection inside the kernel, or from rows; and a long slowly decaying sum."""
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(S + R)
    n = 5
    st = step_of([1] * n, list(range(n)), [3] * n)
    x, low, z = rng.normal(size=(n, C)), rng.normal(size=(n, R + 2 * S)), rng.normal(size=(n, C))
    w, bias, a_log, skip = bf(rng.normal(size=(C, R)) / np.sqrt(R)), rng.normal(size=C) - 1.0, rng.normal(size=(C, S)), rng.normal(size=C)
    state0 = rng.normal(size=(n, 2, C * S))
    want = np.zeros((n, C))
    for i in range(n):
        dt = P.softplus(w @ low[i, :R] + bias)
        Sn = np.exp(dt[:, None] * -np.exp(a_log)) * state0[i, 1].reshape(C, S) + (dt * x[i])[:, None] * low[i, R:R + S][None]
        want[i] = (Sn @ low[i, R + S:] + skip * x[i]) * P.silu(z[i]) * 0.7
    for dtype in (torch.bfloat16, torch.float32):
        for inside in (True, False):
            state, out = dev(state0), torch.empty((n, C), dtype=dtype, device="cuda")
            dt = None if inside else dev(low[:, :R] @ w.T)
            K.selective_scan(dev(x), dev(low), R, S, dev(bias), dev(a_log), dev(skip), dev(z), out, st, state, 0, dt=dt,
                             dt_weight=dev(w, dtype) if inside else None, scale=0.7)
            assert np.abs(out.float().cpu().numpy() - want).max() < (2e-5 if dtype == torch.float32 else 1e-2) * np.abs(want).max()
            assert torch.equal(state[:, 1], dev(state0)[:, 1])          # position 3 reads copy 1 and writes copy 0


def test_a_state_remembers_far_back():
    """A channel that hardly decays: an impulse at the first token is still there two thousand tokens later, in portions too."""
    from burn_lm_b200 import kernels as K
    T, C, S = 2100, 8, 4
    x, z = np.zeros((T, C)), np.full((T, C), 3.0)
    x[0] = 50.0
    low = np.ones((T, 1 + 2 * S))
    a_log, dt = np.full((C, S), np.log(1e-3)), np.full((T, C), -1.0)
    step_size = P.softplus(-1.0)
    last = 50.0 * step_size * S * np.exp(-1e-3 * step_size * (T - 1)) * P.silu(3.0)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        for cuts in ([T], [1, 31, 33, 700, T - 765], [T - 3, 1, 1, 1]):
            state, at, out = torch.full((1, 2, C * S), float("nan"), device="cuda"), 0, None
            for k in cuts:
                st, rows = step_of([k], [0], [at]), slice(at, at + k)
                out = torch.empty((k, C), dtype=dtype, device="cuda")
                K.selective_scan(dev(x[rows]), dev(low[rows]), 1, S, dev(np.zeros(C)), dev(a_log), dev(np.zeros(C)), dev(z[rows]), out, st, state, 0,
                                 dt=dev(dt[rows]))
                at += k
            assert np.abs(out[-1].float().cpu().numpy() - last).max() < tol * last, cuts


@pytest.mark.parametrize("channels,taps", [(64, 4), (33, 3), (40, 2), (24, 1), (20, 6)])
def test_the_convolution_over_rows_of_several_sequences(channels, taps):
    """Long portions slide a window over the rows; it starts anew where a sequence ends, from what the sequence carries."""
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(channels)
    w, b = rng.normal(size=(channels, taps)), rng.normal(size=channels)
    xs = [rng.normal(size=(n, channels)) for n in (150, 3, 70, 1)]
    want = [P.silu(P.convolution(x, w, b)) for x in xs]
    state = torch.full((4, 2, max(1, (taps - 1) * channels)), float("nan"), device="cuda")
    at = [0] * 4
    for portions in ((100, 2, 33, 1), (49, 1, 36, 0), (1, 0, 1, 0)):
        live = [s for s in range(4) if portions[s]]
        st = step_of([portions[s] for s in live], live, [at[s] for s in live])
        x = dev(np.concatenate([xs[s][at[s]:at[s] + portions[s]] for s in live]))
        out, rounded = torch.empty_like(x), torch.empty(x.shape, dtype=torch.bfloat16, device="cuda")
        K.causal_conv(x, 0, channels, dev(w), dev(b), out, 0, st, state, 0, silu=True, out_bf16=rounded)
        exp = np.concatenate([want[s][at[s]:at[s] + portions[s]] for s in live])
        assert np.abs(out.cpu().numpy() - exp).max() < 1e-5 and torch.equal(rounded, out.to(torch.bfloat16))
        at = [a + p for a, p in zip(at, portions)]


# one key made to stand out among hundreds ----------------------------------------------------------------
def planted(n, j, dk, maps, entry_of, gate=False, dv=24):
    """One head; the query reads the first half of the input's lanes and the key the second half, so that the last token's
    query points along the key of token j and along no other token's (its own too); the values are a random map."""
    rng = np.random.default_rng(n + j)
    width = 2 * dk * maps
    entry = entry_of(width)
    half = dk * maps
    zero, eye = np.zeros((half, half)), np.eye(half)
    h = bf(rng.normal(size=(n, width)))
    u = bf(rng.normal(size=half))
    h[n - 1, :half] = u
    h[j, half:] = u
    w = {"q": np.hstack([eye, zero]), "k": np.hstack([zero, eye]), "v": bf(rng.normal(size=(dv, width)) / np.sqrt(width)), "o": np.eye(dv)}
    if gate:
        w["g"] = bf(rng.normal(size=(dv, width)) / np.sqrt(width))
    return entry, width, w, h


FAR = [(300, 0), (300, 1), (300, 63), (300, 64), (300, 127), (300, 298), (65, 0), (129, 64), (2, 0)]


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("dk", [32, 64])
@pytest.mark.parametrize("n,j", FAR)
def test_a_key_far_back_at_page_borders_and_among_the_first_tokens(n, j, dk, decoded, dtype, tol):
    dv = 64 if dk == 64 else 24
    entry, width, w, h = planted(n, j, dk, 1, lambda d: scaled(1, 1, dk, dv, None, rot_dims=0, scaling=None, scale=1.5), dv=dv)
    want = P.full_attention(h, w, entry["mixer"], 1e-5)
    assert np.abs(want[-1] - w["v"] @ h[j]).max() < 1e-2       # the test is sharp: the last token reads token j's value and next to nothing else
    plan = mixer_plan(entry, width)
    part = bound(plan, {"l0.mix." + k: v for k, v in w.items()}, dtype)
    got = run_mixer(part, OwnCache(part, dtype, seed=j), [h], [3], [(n - 1,), (1,)] if decoded else [(n,)], dtype)[0]
    assert np.abs(got[-1] - want[-1]).max() < tol * max(1.0, np.abs(want[-1]).max()) and np.abs(got - want).max() < 3 * tol * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("dtype,tol", [("float32", 2e-4), ("bfloat16", 4e-2)])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("n,j", FAR[:7])
def test_either_map_of_a_head_reads_a_key_far_back(n, j, which, decoded, dtype, tol):
    """The other map's query is zero, so that it averages all values: the head's output is token j's value less a little
    of the mean, or the mean less a little of token j's value."""
    dk, dv = 32, 64
    entry, width, w, h = planted(n, j, dk, 2, lambda d: difference(1, 1, dk, dv, None, rot_dims=0, scale=2.0, diff=0.5), dv=dv)
    keep = np.zeros(2 * dk)
    keep[which * dk:(which + 1) * dk] = 1.0
    w["q"] = w["q"] * keep[:, None]
    w.update(lq1=np.zeros(dk), lk1=np.zeros(dk), lq2=np.zeros(dk), lk2=np.zeros(dk))
    want = P.differential_attention(h, w, entry["mixer"], 1e-5)
    v = h @ w["v"].T
    a = [v[j], v.mean(axis=0)] if which == 0 else [v.mean(axis=0), v[j]]
    assert np.abs(want[-1] - P.rms(a[0] - 0.5 * a[1], 1e-5) * 0.5).max() < 2e-2
    part = bound(mixer_plan(entry, width), {"l0.mix." + k: v for k, v in w.items()}, dtype)
    got = run_mixer(part, OwnCache(part, dtype, seed=j), [h], [3], [(n - 1,), (1,)] if decoded else [(n,)], dtype)[0]
    assert np.abs(got - want).max() < tol * np.abs(want).max()


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 3e-2)])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("dk", [32, 64])
@pytest.mark.parametrize("n,chunk,j", [(300, 75, 225), (300, 75, 224), (226, 75, 225), (227, 75, 225), (227, 75, 224), (300, 64, 256), (300, 64, 255),
                                       (257, 64, 256), (258, 64, 256), (258, 64, 255), (300, 100, 200), (300, 100, 199), (300, 2, 298), (300, 2, 297),
                                       (301, 300, 299), (300, 300, 0), (150, 200, 0), (193, 96, 192), (194, 96, 192), (194, 96, 191), (65, 64, 0)])
def test_a_key_just_inside_and_just_outside_the_chunk(n, chunk, j, dk, decoded, dtype, tol):
    dv = 64 if dk == 64 else 24
    entry, width, w, h = planted(n, j, dk, 1, lambda d: pair(1, 1, dk, dv, chunk, 8, 1, 1, 1, None, rot_dims=0, scale=1.5), gate=True, dv=dv)
    m = entry["mixer"]["left"]
    want = P.chunk_attention(h, w, m)
    gate = P.sigmoid(w["g"] @ h[-1])
    if j < n - 1:
        assert (np.abs(want[-1] - gate * (w["v"] @ h[j])).max() < 1e-2) == ((n - 1) // chunk == j // chunk)       # the test is sharp: all or nothing of token j
    plan = mixer_plan(entry, width).spec.left
    part = bound(plan, {"l0.mix.left." + k: v for k, v in w.items()}, dtype)
    got = run_mixer(part, OwnCache(part, dtype, seed=j), [h], [2], [(n - 1,), (1,)] if decoded else [(n,)], dtype)[0]
    assert np.abs(got[-1] - want[-1]).max() < tol * max(1.0, np.abs(want[-1]).max()) and np.abs(got - want).max() < 3 * tol * max(1.0, np.abs(want).max())


def test_a_negative_scale():
    rng = np.random.default_rng(11)
    for entry, plain in ((scaled(4, 2, 32, 40, None, scale=-0.4), lambda h, w, m: P.full_attention(h, w, m, 1e-5)),
                         (difference(2, 1, 64, 128, None, scale=-0.2), lambda h, w, m: P.differential_attention(h, w, m, 1e-5))):
        for dtype, tol in (("float32", 5e-5), ("bfloat16", 4e-2)):
            check_mixer(entry, plain, 64, (150,), [1], [(100,), (30,)] + [(1,)] * 20, dtype, tol, 3)


# the stream, the feed-forwards ----------------------------------------------------------------------------
def test_the_stream_at_the_start_of_a_pass():
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(2)
    n, d = 37, 72
    x, a, e, v = (rng.normal(size=s) for s in ((n, d), (n, d), (n, d), (d,)))
    for delta in (None, torch.float32, torch.bfloat16):
        for again in (False, True):
            resid, dl = dev(x), dev(a, delta) if delta is not None else None
            K.pass_entry(resid, dl, dev(e) if again else None, dev(v))
            want = x + (dl.double().cpu().numpy() if dl is not None else 0.0) + (e if again else 0.0) + v
            assert np.abs(resid.cpu().numpy() - want).max() < 1e-5


@pytest.mark.parametrize("around_zero", [True, False])
def test_norm_weights_around_zero(around_zero):
    from burn_lm_b200.parts.base import Runtime
    from burn_lm_b200.parts.norm import RMSNorm, RMSNormSpec
    rng = np.random.default_rng(3)
    x, w = rng.normal(size=(9, 64)), bf(0.3 * rng.normal(size=64))
    norm = RMSNorm(RMSNormSpec(64, 1e-3, around_zero=around_zero), {"weight": "w"}, Runtime(torch.float32, torch.device("cuda")))
    norm.bind({"w": dev(w, torch.bfloat16)})
    got = norm.add_norm(dev(x), None).cpu().numpy()
    assert np.abs(got - P.rms(x, 1e-3) * (w + (1.0 if around_zero else 0.0))).max() < 1e-5


@pytest.mark.parametrize("dtype,tol", [("float32", 2e-5), ("bfloat16", 2e-2)])
@pytest.mark.parametrize("n,width,ff", [(1, 64, 128), (8, 128, 200), (16, 320, 72), (17, 64, 96), (200, 72, 100), (1100, 128, 264), (1030, 200, 50), (5, 36, 20)])
def test_squared_relu_feed_forward(n, width, ff, dtype, tol):
    """Every route: the skinny product, the library's, the tcgen05 product, the 32-bit one."""
    from burn_lm_b200.parts.base import Runtime
    from burn_lm_b200.parts.feed_forward import MLP, MLPSpec
    rng = np.random.default_rng(n)
    x, up, down = bf(rng.normal(size=(n, width))), bf(rng.normal(size=(ff, width)) / np.sqrt(width)), bf(rng.normal(size=(width, ff)) / np.sqrt(ff))
    part = MLP(MLPSpec(width, ff), {"up": "u", "down": "d"}, Runtime(DTYPES[dtype], torch.device("cuda")))
    part.bind({"u": dev(up, DTYPES[dtype]), "d": dev(down, DTYPES[dtype])})
    got = part.forward(dev(x, DTYPES[dtype]), SimpleNamespace(handoff=None)).float().cpu().numpy()
    want = P.dense(x, up, down)
    assert np.abs(got - want).max() < tol * np.abs(want).max()


@pytest.mark.parametrize("n_experts,top", [(12, 3), (8, 2), (5, 5), (4, 1), (1, 1), (33, 4)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_routing_by_logits_with_a_bias(n_experts, top, dtype):
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(n_experts + top)
    h, router, bias = bf(rng.normal(size=(45, 40))), bf(8.0 * rng.normal(size=(n_experts, 40)) / np.sqrt(40)), bf(2.0 * rng.normal(size=n_experts))
    want_ids, want_w = P.route(h, router, bias, top)
    ids, weights = K.moe_route(dev(h, dtype), dev(router), top, scores=K.SCORES_CHOSEN_SOFTMAX, bias=dev(bias))
    assert np.array_equal(ids.cpu().numpy(), want_ids) and np.allclose(weights.cpu().numpy(), want_w, atol=1e-5)
    if n_experts > 1 and top < n_experts:
        assert not np.array_equal(P.route(h, router, np.zeros(n_experts), top)[0], want_ids)      # the bias matters
    # logits far apart (a softmax over all of them would underflow): the choice still goes by the logits
    ids, weights = K.moe_route(dev(h, dtype), dev(router), top, scores=K.SCORES_CHOSEN_SOFTMAX, bias=dev(300.0 * np.arange(n_experts)))
    assert ids.cpu().numpy().tolist() == [[n_experts - 1 - k for k in range(top)]] * 45 and np.allclose(weights.cpu().numpy()[:, 0], 1.0)


@pytest.mark.parametrize("n,width,ff,n_experts,top", [(3, 64, 48, 6, 2), (45, 40, 24, 8, 2), (150, 36, 20, 6, 2), (60, 72, 40, 1, 1), (70, 128, 256, 6, 2),
                                                      (700, 136, 72, 4, 2), (1100, 64, 264, 3, 1), (520, 128, 128, 2, 2)])
def test_squared_relu_experts(n, width, ff, n_experts, top):
    """Every route of the experts' products: CUDA cores, mma.sync tiles of 16 and 64 places, tcgen05."""
    from burn_lm_b200 import kernels as K
    rng = np.random.default_rng(n)
    h, router, bias = bf(rng.normal(size=(n, width))), bf(rng.normal(size=(n_experts, width))), 20.0 * rng.permutation(n_experts).astype(np.float64)
    w = {"router": router, "router.b": bias}
    for e in range(n_experts):
        w[f"e{e}.up"], w[f"e{e}.down"] = bf(1.5 * rng.normal(size=(ff, width)) / np.sqrt(width)), bf(rng.normal(size=(width, ff)) / np.sqrt(ff))
    want = P.experts(h, w, experts(n_experts, top, ff))
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
        ids, weights = K.moe_route(dev(h, dtype), dev(router), top, scores=K.SCORES_CHOSEN_SOFTMAX, bias=dev(bias))
        up, down = (dev(np.stack([w[f"e{e}.{r}"] for e in range(n_experts)]), dtype) for r in ("up", "down"))
        got = K.moe_experts(dev(h, dtype), ids, weights, up, down, weight_on_input=False, out_dtype=torch.float32, unit=K.UNIT_RELU2)
        assert np.abs(got.cpu().numpy() - want).max() < tol * np.abs(want).max()


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
            seen.append((resid if pending is None else resid + pending).cpu().numpy())      # what the layer's last sublayer left joins the stream
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


@pytest.mark.parametrize("name", ["tom_a", "tom_c", "tom_d"])
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
    folder = make_folder(tmp_path, "tom_a")
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


@pytest.mark.parametrize("name", ["tom_a", "tom_c"])
def test_long_decoding_while_the_chunks_give_pages_back(tmp_path, name):
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
    chunked = [g for g in engine.cache._kv_groups if g.need.chunk]
    assert chunked and all(len(g.live_pages(slot)) <= (g.need.chunk + PAGE - 1) // PAGE + 1 for g in chunked)
    engine.release(slot)
    engine.verify()


@pytest.mark.parametrize("name", ["tom_a", "tom_b"])
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
    folder = make_folder(tmp_path, "tom_a")
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
    folder = make_folder(tmp_path, "tom_a")
    lm = blm.load(folder, dtype="bfloat16", max_seq_len=256, max_batch=2)
    prompts = [random_tokens(50, 20, 272), random_tokens(51, 66, 272)]
    a = lm.generate(prompts, sample_len=12, temperature=0.8, seed=7, ignore_stop=True).tokens
    b = lm.generate(prompts, sample_len=12, temperature=0.8, seed=7, ignore_stop=True).tokens
    assert a == b and all(len(t) == 12 for t in a)          # the same draws from the same seed, through used slots


def test_the_trace_runner_as_a_child_process(tmp_path):
    cfg = CONFIGS["tom_c"]
    a, b = random_tokens(40, 115, cfg["vocab"]), random_tokens(41, 9, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:110], "want": [0, 109]}, {"id": "b", "tokens": b[:5], "want": [4]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[110]], "want": []}, {"id": "b", "tokens": [b[5]], "want": [0]}], "end": []}]
    steps += [{"step": 2 + t, "entries": [{"id": "a", "tokens": [a[111 + t]], "want": [0]}] + ([{"id": "b", "tokens": [b[6 + t]], "want": [0]}] if t < 3 else []),
               "end": ["b"] if t == 2 else []} for t in range(4)]
    out = tmp_path / "out"
    for dtype, tol in (("float32", FP32_TOL), ("bfloat16", BF16_TOL)):
        folder = folder_for(tmp_path, "tom_c", dtype)
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
    r = subprocess.run(program + ["random", folder, "--preset", "tomalix_tiny", "--seed", "4", "--dtype", "float32"],
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


@pytest.mark.parametrize("kinds", ["differences only", "pairs only", "scaled only, no feed-forward", "no loop, pairs first and last", "the whole model loops"])
def test_models_of_one_kind_of_layer_and_other_orders(tmp_path, kinds):
    e, d = experts(6, 2, 32), dense(72)
    layers, loop = {
        "differences only": ([difference(4, 2, 16, 24, e, rot_dims=8), difference(2, 2, 24, 24, None)], None),
        "pairs only": ([pair(2, 1, 16, 24, 50, 40, 6, 4, 5, d), pair(3, 3, 8, 16, 7, 64, 16, 2, 4, None, rot_dims=4)], (1, 2, 3)),
        "scaled only, no feed-forward": ([scaled(2, 1, 24, 16, None), scaled(3, 3, 8, 16, None, rot_dims=0), scaled(1, 1, 64, 64, None)], (0, 2, 2)),
        "no loop, pairs first and last": ([pair(2, 2, 16, 16, 64, 32, 8, 4, 4, e), scaled(2, 1, 16, 16, d), difference(4, 4, 8, 8, e), pair(1, 1, 16, 48, 128, 48, 3, 3, 8, d)], None),
        "the whole model loops": ([difference(2, 1, 16, 16, d), pair(2, 1, 16, 32, 30, 64, 4, 4, 4, e)], (0, 2, 4)),
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
