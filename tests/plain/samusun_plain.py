"""Plain, slow implementation of the Samusun decoder: whole sequences, no cache, no batching.

One function per mechanism, numpy float64 throughout, written from the design's equations and
sharing no code with the product package (model folders are read with the `safetensors` package).

Notation: x is the residual stream [T, D]; h the one normed input that both parts of a layer read; H query heads on G
key/value heads of d lanes; S [d, e] the state of a retention head with e value lanes.
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
def silu(z):
    return z / (1.0 + np.exp(-z))


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


# --------------------------------------------------------------------------------------------
# attention: keys that are their own values, a bias by distance, queries scaled by position
# --------------------------------------------------------------------------------------------
def query_temperature(positions, coef, every):
    """1 + coef ln(floor((p + 1) / every) + 1), a number per position."""
    return np.array([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in positions])


def slopes(n_heads):
    """What a step of distance costs every head."""
    return np.array([2.0 ** (-8.0 * (h + 1) / n_heads) for h in range(n_heads)])


def sliding_window(T, size):
    """[T, T]: which of the keys j a query i sees: the latest `size` up to its own."""
    i = np.arange(T)
    back = i[:, None] - i[None, :]
    return (back >= 0) & (back < size)


def biased_scores(q, k, scale, slope):
    """[T, T] of one head: scale q.k less the distance times the head's slope."""
    i = np.arange(q.shape[0])
    return scale * (q @ k.T) - slope * (i[:, None] - i[None, :])


def shared_attention(q, k, scale, seen):
    """q [T, H, d], k [T, G, d] -> [T, H, d]; head h reads key/value head h // (H / G), whose keys are the values."""
    T, H, d = q.shape
    share = H // k.shape[1]
    slope, out = slopes(H), np.empty((T, H, d))
    for h in range(H):
        keys = k[:, h // share]
        s = np.where(seen, biased_scores(q[:, h], keys, scale, slope[h]), -np.inf)
        out[:, h] = softmax(s) @ keys
    return out


def attention(h, w, m):
    T = h.shape[0]
    q = (h @ w["q"].T + w["q.b"]).reshape(T, m["heads"], m["dim"])
    k = (h @ w["k"].T + w["k.b"]).reshape(T, m["kv_heads"], m["dim"])
    temp = m.get("q_temp")
    if temp:
        q = q * query_temperature(range(T), temp["coef"], temp["every"])[:, None, None]
    size = m["mask"]["size"] if m.get("mask") else T
    a = shared_attention(q, k, m["scale"], sliding_window(T, size))
    return a.reshape(T, -1) @ w["o"].T + w["o.b"]


# --------------------------------------------------------------------------------------------
# retention
# --------------------------------------------------------------------------------------------
def rotate_halves(x, positions, dims, base):
    """x [T, ..., d]: a turn of lanes (i, i + dims / 2) by position * base^(-2i / dims); lanes from dims on stay."""
    if dims == 0:
        return x.copy()
    half = dims // 2
    freq = np.array([base ** (-2.0 * i / dims) for i in range(half)])
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (half,)
    c, s = np.cos(ang).reshape(shape), np.sin(ang).reshape(shape)
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def retain(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, e], a decay per head: S <- decay S + k v^T, o = S^T q.  Returns (o [T, H, e], last S)."""
    T, H, d = q.shape
    e = v.shape[-1]
    S = np.zeros((H, d, e)) if state is None else state.copy()
    out = np.empty((T, H, e))
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    return out, S


def retention(h, w, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    turn = lambda x: rotate_halves(x.reshape(T, H, d), range(T), rot["dims"], rot["base"])
    q, k, v = turn(h @ w["q"].T), turn(h @ w["k"].T) * d ** -0.5, (h @ w["v"].T).reshape(T, H, e)
    o, _ = retain(q, k, v, np.asarray(m["decay"], dtype=np.float64))
    return (rms(o, eps).reshape(T, H * e) * silu(h @ w["g"].T)) @ w["o"].T


# --------------------------------------------------------------------------------------------
# feed-forwards
# --------------------------------------------------------------------------------------------
def dense(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, top):
    """(chosen experts [T, top], their scores [T, top]): a softmax over all experts, of which the largest are kept as they are."""
    s = softmax(h @ router.T)
    order = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return order, np.take_along_axis(s, order, axis=-1)


def experts(h, w, f):
    ids, weights = route(h, w["router"], f["router"]["top"])
    out = np.zeros_like(h)
    for e in range(f["router"]["experts"]):
        for t, k in zip(*np.nonzero(ids == e)):
            out[t] += weights[t, k] * dense(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    return out


def feed_forward(h, w, f):
    return dense(h, w["gate"], w["up"], w["down"]) if f["kind"] == "dense" else experts(h, w, f)


# --------------------------------------------------------------------------------------------
# the model
# --------------------------------------------------------------------------------------------
def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def mixer(h, kind, w, m, eps):
    if kind == "attention":
        return attention(h, w, m)
    if kind == "retention":
        return retention(h, w, m, eps)
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


def forward(cfg, tensors, tokens, after=None):
    """Logits [T, vocab] of a whole sequence; `after`: a list that receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = tensors["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, t in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + tensors["loop.step"][t]
        h = rms_norm(x, tensors[p + "norm1"], eps)
        both = mixer(h, layer["type"], sub(tensors, p + "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            both = both + feed_forward(h, sub(tensors, p + "mlp."), layer["mlp"])
        x = x + both
        if after is not None:
            after.append(x.copy())
    logits = rms_norm(x, tensors["final.norm"], eps) @ tensors["head"].T * cfg.get("logit_scale", 1.0)
    return soft_cap(logits, cfg.get("logit_softcap"))


def greedy(cfg, tensors, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(np.argmax(forward(cfg, tensors, tokens)[-1])))
    return tokens[len(prompt):]
