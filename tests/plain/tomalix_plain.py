"""Plain, slow implementation of the Tomalix decoder: whole sequences, no cache, no batching.

One function per mechanism, numpy float64 throughout, written from the design's equations and
sharing no code with the product package (model folders are read with the `safetensors` package).

Notation: x is the residual stream [T, D]; h the input of a mixer; H query heads on G key/value heads, dk the
query/key size of a head (of one map of it where a head has two), dv its value size; C the channels and S the states
a channel of the selective scan.
"""
from __future__ import annotations

import json
import math
import os

import numpy as np


def read_model_folder(folder):
    """config.json as a dict and every tensor as float64 (integer tables as int64), by stored name."""
    import torch
    from safetensors.torch import load_file

    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    raw = load_file(os.path.join(folder, "model.safetensors"))
    tensors = {k: (v.to(torch.float64).numpy() if v.is_floating_point() else v.to(torch.int64).numpy())
               for k, v in raw.items()}
    return cfg, tensors


# --------------------------------------------------------------------------------------------
# small functions
# --------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def squared_relu(z):
    return np.square(np.maximum(z, 0.0))


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    """The stored weight is what the multiplier exceeds 1 by."""
    return rms(x, eps) * (1.0 + w)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


# --------------------------------------------------------------------------------------------
# positions
# --------------------------------------------------------------------------------------------
def plain_frequencies(rot):
    return np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])


def linear_frequencies(rot):
    """(frequencies, multiplier of cosine and sine): every frequency divided by the factor."""
    s = rot.get("scaling")
    return plain_frequencies(rot) / (s["factor"] if s else 1.0), 1.0


def yarn_frequencies(rot):
    """Frequencies between the plain ones (lanes that turn often) and the divided ones (lanes that turn seldom)."""
    f, s = plain_frequencies(rot), rot.get("scaling")
    if not s:
        return f, 1.0
    dims = rot["dims"]

    def lane(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))

    lo = max(math.floor(lane(s["fast"])), 0)
    hi = min(math.ceil(lane(s["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate_halves(x, positions, dims, freq, mult=1.0):
    """x [T, ..., d]: lanes i and i + dims / 2 turn together by position * freq[i]; lanes from dims on pass."""
    if dims == 0:
        return x.copy()
    half = dims // 2
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (half,)
    c, s = mult * np.cos(ang).reshape(shape), mult * np.sin(ang).reshape(shape)
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


# --------------------------------------------------------------------------------------------
# attention
# --------------------------------------------------------------------------------------------
def causal(T):
    i = np.arange(T)
    return i[None, :] <= i[:, None]


def chunked(T, size):
    i = np.arange(T)
    return causal(T) & (i[None, :] // size == i[:, None] // size)


def attend(q, k, v, scale, visible):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]."""
    share = q.shape[1] // k.shape[1]
    k, v = np.repeat(k, share, axis=1), np.repeat(v, share, axis=1)
    s = np.einsum("thd,shd->hts", q, k) * scale
    p = softmax(np.where(visible[None], s, -np.inf))
    return np.einsum("hts,shd->thd", p, v)


def grouped_attention(h, w, m, turning, visible):
    """The heads' outputs [T, H, dv], before gate and output projection; turning: (frequencies, multiplier)."""
    T = h.shape[0]
    pos = np.arange(T)
    q = (h @ w["q"].T).reshape(T, m["heads"], m["dim"])
    k = (h @ w["k"].T).reshape(T, m["kv_heads"], m["dim"])
    v = (h @ w["v"].T).reshape(T, m["kv_heads"], m["vdim"])
    q = rotate_halves(q, pos, m["rot"]["dims"], *turning)
    k = rotate_halves(k, pos, m["rot"]["dims"], *turning)
    return attend(q, k, v, m["scale"], visible)


def full_attention(h, w, m, eps):
    """Causal, with the frequencies blended (YaRN)."""
    o = grouped_attention(h, w, m, yarn_frequencies(m["rot"]), causal(h.shape[0]))
    return o.reshape(h.shape[0], -1) @ w["o"].T


def chunk_attention(h, w, m):
    """Inside chunks of the sequence, with a gate on every lane of the heads' outputs."""
    o = grouped_attention(h, w, m, (plain_frequencies(m["rot"]), 1.0), chunked(h.shape[0], m["mask"]["size"]))
    return (o.reshape(h.shape[0], -1) * sigmoid(h @ w["g"].T)) @ w["o"].T


def difference_weight(w, diff):
    return math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    """[T, H, dv] each."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, w, m, eps):
    """Two maps a head over the same values; causal, with every frequency divided."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, turning = np.arange(T), linear_frequencies(m["rot"])
    q = rotate_halves((h @ w["q"].T).reshape(T, H, 2, dk), pos, m["rot"]["dims"], *turning)
    k = rotate_halves((h @ w["k"].T).reshape(T, G, 2, dk), pos, m["rot"]["dims"], *turning)
    v = (h @ w["v"].T).reshape(T, G, dv)
    a = [attend(q[:, :, i], k[:, :, i], v, m["scale"], causal(T)) for i in (0, 1)]
    o = difference_of_maps(a[0], a[1], difference_weight(w, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * dv) @ w["o"].T


# --------------------------------------------------------------------------------------------
# the selective scan
# --------------------------------------------------------------------------------------------
def convolution(x, taps, bias):
    """x [T, C], taps [C, K]: bias + sum_j taps[:, j] x_(t - (K - 1) + j), zeros before the start."""
    T, C = x.shape
    K = taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, C)), x], axis=0)
    y = np.zeros((T, C)) + bias
    for j in range(K):
        y += padded[j:j + T] * taps[:, j]
    return y


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, C], A [C, S], B, C [T, S], D [C]: S <- exp(dt A) S + dt x B;  y = S C + D x."""
    S = np.zeros(A.shape)
    out = np.zeros(x.shape)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba(h, w, m):
    inner, rank, S = m["inner"], m["dt_rank"], m["state"]
    both = h @ w["in"].T
    x, z = both[:, :inner], both[:, inner:]
    x = silu(convolution(x, w["conv"], w["conv.b"]))
    low = x @ w["x"].T
    dt = softplus(low[:, :rank] @ w["dt"].T + w["dt.b"])
    y = selective_scan(x, dt, -np.exp(w["A_log"]), low[:, rank:rank + S], low[:, rank + S:], w["D"])
    return (y * silu(z)) @ w["o"].T


def parallel_mixers(h, w, m):
    left = chunk_attention(h, sub(w, "left."), m["left"])
    right = mamba(h, sub(w, "right."), m["right"])
    return m["left_scale"] * left + m["right_scale"] * right


# --------------------------------------------------------------------------------------------
# feed-forward
# --------------------------------------------------------------------------------------------
def dense(h, up, down):
    return squared_relu(h @ up.T) @ down.T


def route(h, router, bias, top):
    """(chosen experts [T, top], their weights [T, top])."""
    z = h @ router.T + bias
    order = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    return order, softmax(np.take_along_axis(z, order, axis=-1))


def experts(h, w, f):
    ids, weights = route(h, w["router"], w["router.b"], f["router"]["top"])
    out = np.zeros_like(h)
    for e in range(f["router"]["experts"]):
        for t, k in zip(*np.nonzero(ids == e)):
            out[t] += weights[t, k] * dense(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    return out


def feed_forward(h, w, f):
    return dense(h, w["up"], w["down"]) if f["kind"] == "dense" else experts(h, w, f)


# --------------------------------------------------------------------------------------------
# the model
# --------------------------------------------------------------------------------------------
def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def mixer(h, kind, w, m, eps):
    if kind == "attention":
        return differential_attention(h, w, m, eps)
    if kind == "attention_2":
        return full_attention(h, w, m, eps)
    if kind == "parallel":
        return parallel_mixers(h, w, m)
    raise ValueError(kind)


def run_order(cfg):
    """[(layer, number of the pass that starts with this run or None)]."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def before_pass(x, x0, steps, t):
    if t > 0:
        x = x + x0
    return x + steps[t]


def forward(cfg, tensors, tokens, after=None):
    """Logits [T, vocab] of a whole sequence; `after`: a list that receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = tensors["embed"][np.asarray(tokens)]
    x = x0.copy()
    for i, t in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = before_pass(x, x0, tensors["loop.step"], t)
        h = rms_norm(x, tensors[p + "norm1"], eps)
        x = x + mixer(h, layer["type"], sub(tensors, p + "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + feed_forward(rms_norm(x, tensors[p + "norm2"], eps), sub(tensors, p + "mlp."), layer["mlp"])
        if after is not None:
            after.append(x.copy())
    logits = rms_norm(x, tensors["final.norm"], eps) @ tensors["head"].T
    return soft_cap(logits, cfg.get("logit_softcap"))


def greedy(cfg, tensors, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(np.argmax(forward(cfg, tensors, tokens)[-1])))
    return tokens[len(prompt):]
