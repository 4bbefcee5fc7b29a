"""Small configurations of the Tomalix decoder for the tests, differing in every size and option, with helpers.

The folders are written here, not by the package's random-weights mode: matrices are drawn with a spread of
gain / sqrt(inputs), so that attention weights are far from equal, the two maps of a head differ, gates and step sizes
spread over their range and the router decides clearly; a fault in a rotation, a chunk, a state or a choice of experts
then moves the logits by far more than rounding does.
"""
import json
import os

import numpy as np

from burn_lm_b200.config import preset


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}


def rotation(dims, base, scaling=None):
    rot = {"dims": dims, "base": base}
    if scaling is not None:
        rot["scaling"] = {"factor": scaling} if isinstance(scaling, float) else dict(zip(("factor", "original", "fast", "slow"), scaling))
    return rot


def difference(heads, kv_heads, dim, vdim, mlp, rot_dims=None, base=10000.0, factor=2.0, scale=None, diff=0.4):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "diff": diff,
                      "rot": rotation(dim if rot_dims is None else rot_dims, base, factor)}}


def scaled(heads, kv_heads, dim, vdim, mlp, rot_dims=None, base=10000.0, scaling=(4.0, 128, 16.0, 1.0), scale=None):
    return {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                      "rot": rotation(dim if rot_dims is None else rot_dims, base, scaling)}}


def pair(heads, kv_heads, dim, vdim, chunk, inner, state, conv, dt_rank, mlp, rot_dims=None, base=10000.0, scale=None, scales=(0.7, 0.55)):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                               "mask": {"size": chunk}, "rot": rotation(dim if rot_dims is None else rot_dims, base)},
                      "right": {"inner": inner, "state": state, "conv": conv, "dt_rank": dt_rank},
                      "left_scale": scales[0], "right_scale": scales[1]}}


def model(vocab, width, layers, loop=None, cap=None, eps=1e-5):
    cfg = {"architecture": "Tomalix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap is not None:
        cfg["logit_softcap"] = cap
    return cfg


# every branch (see the preset)
TOM_A = preset("tomalix_tiny")
# values that a model may happen to make equal or 1: one head everywhere, keys as wide as values, one expert, as many chosen
# as there are, one chosen, one tap (nothing carried), one state, a rank of one, chunks of one and of two tokens, scales of
# 1, a factor of 1, no turning lane, a loop that runs once over the first layer, no cap
TOM_B = model(131, 64, [
    difference(1, 1, 32, 32, experts(1, 1, 64), scale=1.0, factor=1.0, diff=0.0),
    pair(1, 1, 32, 32, 1, 64, 1, 1, 1, experts(3, 3, 32), scale=1.0, scales=(1.0, 1.0)),
    scaled(1, 1, 16, 16, experts(4, 1, 48), scaling=(1.0, 64, 1.0, 1.0)),
    pair(2, 2, 16, 16, 2, 32, 2, 2, 2, None, rot_dims=0),
    scaled(2, 2, 16, 16, dense(64), rot_dims=0, scaling=None),
], loop=(0, 1, 1))
# sizes that are no multiples of 8 or of a warp: five heads on one key/value head, heads of 12 and 20 lanes of which some
# turn, 44 channels of 5 states with 5 taps and a rank of 3, a width of 72, chunks of 33; the whole model runs three times
TOM_C = model(257, 72, [
    pair(5, 1, 12, 20, 33, 44, 5, 5, 3, experts(5, 3, 40), rot_dims=6, base=500.0, scale=0.31),
    difference(5, 1, 12, 20, dense(100), rot_dims=6, base=500.0, factor=3.0, diff=0.7),
    scaled(3, 3, 20, 12, None, rot_dims=10, base=300.0, scaling=(6.0, 50, 9.0, 1.5), scale=0.3),
    difference(3, 3, 20, 20, experts(7, 2, 24), rot_dims=4, diff=0.25),
], loop=(0, 4, 3), cap=12.0, eps=1e-6)
# heads of 64 and 128 lanes, values of 128 and 256, two to eight query heads a key/value head, 16 and 40 states, chunks
# beyond two pages: the sizes of large models; the loop is the last layers
TOM_D = model(300, 128, [
    difference(4, 2, 64, 128, experts(16, 4, 64), base=1e6, diff=0.5),
    scaled(4, 1, 128, 128, dense(256), base=1e6, scaling=(16.0, 4096, 32.0, 1.0)),
    pair(8, 1, 64, 64, 150, 256, 16, 4, 16, dense(192), rot_dims=32),
    scaled(2, 2, 64, 64, experts(8, 2, 128), rot_dims=32),
    pair(2, 1, 128, 256, 200, 128, 40, 4, 8, None, rot_dims=64),
    difference(2, 1, 128, 256, None, rot_dims=32),
], loop=(4, 6, 2), cap=50.0)

CONFIGS = {"tom_a": TOM_A, "tom_b": TOM_B, "tom_c": TOM_C, "tom_d": TOM_D}


def values(rng, name, shape, lively=True):
    """A tensor's values by its stored name's ending; not `lively`: every matrix with a gain of one and router biases two
    apart, which decide the choice of experts alone, for the comparisons in bfloat16, where a close call between two experts
    would otherwise be decided by rounding."""
    last = name.split(".")[-1]
    if last in ("norm", "norm1", "norm2"):
        return 0.2 * rng.normal(size=shape)                      # stored around zero
    if name == "loop.step":
        return 0.5 * rng.normal(size=shape)
    if last in ("lq1", "lk1", "lq2", "lk2"):
        return 0.8 * rng.normal(size=shape) / np.sqrt(shape[0]) ** 0.5
    if name.endswith("router.b"):
        return 0.5 * rng.normal(size=shape) if lively else 2.0 * rng.permutation(shape[0])
    if name.endswith("dt.b"):
        return rng.uniform(-4.0, 0.5, size=shape)                # step sizes from 0.02 to 1
    if name.endswith("conv.b"):
        return 0.3 * rng.normal(size=shape)
    if last == "conv":
        return 0.6 * rng.normal(size=shape)
    if last == "A_log":
        return rng.uniform(-2.0, 2.0, size=shape)
    if last == "D":
        return 1.0 + 0.3 * rng.normal(size=shape)
    if name == "embed":
        return rng.normal(size=shape)
    gain = {"router": 3.0, "q": 2.0, "k": 2.0, "up": 1.5, "g": 2.0, "in": 1.5, "x": 1.5, "dt": 1.5}.get(last, 1.0) if lively else 1.0
    if last == "router" and not lively:
        gain = 0.2
    return gain * rng.normal(size=shape) / np.sqrt(shape[-1])


def make_folder(tmp_path, name, seed=0, config=None, lively=True):
    """A model folder for CONFIGS[name] (or `config`), stored in bfloat16."""
    import torch
    from safetensors.torch import save_file
    from burn_lm_b200.model import tensor_specs_of

    cfg = config if config is not None else CONFIGS[name]
    folder = os.path.join(str(tmp_path), f"{name}-{seed}-{'lively' if lively else 'calm'}")
    if os.path.exists(os.path.join(folder, "model.safetensors")):
        return folder
    os.makedirs(folder, exist_ok=True)
    rng = np.random.default_rng(seed)
    tensors = {}
    for spec in tensor_specs_of(cfg):
        tensors[spec.name] = torch.tensor(values(rng, spec.name, tuple(spec.shape), lively), dtype=torch.float32).to(torch.bfloat16).contiguous()
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(tensors, os.path.join(folder, "model.safetensors"))
    return folder


def random_tokens(seed, n, vocab):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, size=n)]


def row_error(got, want):
    """max |got - want| of every row, relative to the row's largest |want|."""
    got = np.asarray(got, dtype=np.float64)
    want = np.asarray(want, dtype=np.float64)
    return np.abs(got - want).max(axis=-1) / np.abs(want).max(axis=-1)
