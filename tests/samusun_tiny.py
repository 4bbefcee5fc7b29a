"""Small configurations of the Samusun decoder for the tests, differing in every size and option, with helpers.

The folders are written here, not by the package's random-weights mode: matrices are drawn with a spread of
gain / sqrt(inputs), so that attention weights are far from equal, gates spread over their range and the router decides
clearly; a fault in a window, a slope, a temperature, a state or a choice of experts then moves the logits by far more than
rounding does.
"""
import json
import os

import numpy as np

from burn_lm_b200.config import preset


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}


def window(heads, kv_heads, dim, size, mlp, scale=None, q_temp=(0.3, 20)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or 1.5 * dim ** -0.5}
    if size is not None:
        m["mask"] = {"size": size}
    if q_temp is not None:
        m["q_temp"] = dict(zip(("coef", "every"), q_temp))
    return {"type": "attention", "mixer": m, "mlp": mlp}


def retain(heads, dim, vdim, mlp, decay=None, rot_dims=None, base=10000.0):
    decay = decay or [1.0 - 2.0 ** -(2.0 + 6.0 * h / heads) for h in range(heads)]
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}
    if rot_dims != 0:
        m["rot"] = {"dims": dim if rot_dims is None else rot_dims, "base": base}
    return {"type": "retention", "mixer": m, "mlp": mlp}


def model(vocab, width, layers, loop=None, cap=None, eps=1e-5, embed=1.0, logit_scale=1.0):
    cfg = {"architecture": "Samusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
           "logit_scale": logit_scale, "layers": layers}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap is not None:
        cfg["logit_softcap"] = cap
    return cfg


# every branch (see the preset)
SAM_A = preset("samusun_tiny")
# values that a model may happen to make equal or 1: one head everywhere, one expert, as many chosen as there are, one chosen,
# windows of one and two tokens and none, scales of 1, a temperature that steps at every position and one that never moves, a
# decay of one and of nothing, no turning lane, one value lane, a loop that runs once over the first layer, no cap
SAM_B = model(131, 64, [
    window(1, 1, 32, 1, experts(1, 1, 64), scale=1.0, q_temp=(0.5, 1)),
    retain(1, 32, 32, experts(3, 3, 32), decay=[1.0], rot_dims=0),
    window(1, 1, 16, 2, experts(4, 1, 48), q_temp=(0.0, 7)),
    retain(2, 16, 1, dense(64), decay=[0.0, 0.5], rot_dims=2),
    window(2, 2, 16, None, None, q_temp=None),
    retain(2, 16, 16, None, decay=[0.9, 0.9]),
], loop=(0, 1, 1))
# sizes that are no multiples of 8 or of a warp: five heads on one key/value head, heads of 12 and 20 lanes of which some turn,
# values of 7 and 36, a width of 72, windows of 33 and 65; the whole model runs three times
SAM_C = model(257, 72, [
    retain(5, 12, 20, dense(100), rot_dims=6, base=500.0),
    window(5, 1, 12, 33, experts(5, 3, 40), scale=0.31),
    window(3, 3, 20, 65, dense(60), q_temp=(-0.1, 13)),
    retain(3, 20, 7, experts(7, 2, 24), rot_dims=10, base=300.0),
    retain(2, 18, 36, None, decay=[0.999, 0.5], rot_dims=18),
], loop=(0, 5, 3), cap=12.0, eps=1e-6, embed=0.6, logit_scale=0.5)
# heads of 64, 88 and 128 lanes, two to eight query heads a key/value head, windows beyond two pages and of exactly one, wide
# retention heads: the sizes of large models; the loop is the last layers
SAM_D = model(300, 128, [
    window(4, 2, 64, 150, dense(256)),
    retain(2, 64, 128, experts(16, 4, 64), base=1e6),
    window(8, 1, 128, 64, dense(192), scale=0.05),
    retain(1, 256, 200, dense(64), decay=[0.9995], rot_dims=64),
    window(2, 2, 88, 129, experts(8, 2, 128)),
    retain(2, 128, 64, dense(128), decay=[0.97, 0.998]),
], loop=(4, 6, 2), cap=50.0, embed=2.0)

CONFIGS = {"sam_a": SAM_A, "sam_b": SAM_B, "sam_c": SAM_C, "sam_d": SAM_D}


def values(rng, name, shape, lively=True):
    """A tensor's values by its stored name's ending; not `lively`: every matrix with a gain of one and routers that decide by a
    wide margin, for the comparisons in bfloat16, where a close call between two experts would otherwise be decided by rounding."""
    last = name.split(".")[-1]
    if last in ("norm", "norm1"):
        return 1.0 + 0.2 * rng.normal(size=shape)
    if name == "loop.step":
        return 0.5 * rng.normal(size=shape)
    if last == "b":
        return 0.4 * rng.normal(size=shape)
    if name == "embed":
        return rng.normal(size=shape)
    gain = {"router": 3.0, "q": 2.0, "k": 1.5, "up": 1.5, "gate": 1.5, "g": 2.0}.get(last, 1.0) if lively else 1.0
    if last == "router" and not lively:
        gain = 6.0
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
