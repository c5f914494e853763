"""A plain, slow Gararax in float64 numpy: whole sequences, no cache, one function per mechanism.

It shares no code with the package: it reads config.json's keys itself and takes tensors by their checkpoint names.
Notation: T tokens, W the model's width; rows of a [T, n] array are tokens. Weights are [out, in], applied as y = x M^T.

The stream starts as rows of the token table (s0). With r = residual_mult and u(x) = x / sqrt(mean x^2 + eps), a layer is

    s = s + r u(mixer(u(s) w1)) w1b
    s = s + r u(ff(u(s) w2)) w2b                            (layers with a feed-forward)
    s = s + r u(P (gelu(G s) * e_i[token])) w_side          e_i: the layer's columns of a second token table

A span of layers may run several times in a row: pass t starts from s + step[t], and from the second pass on s0 is added
too. Every mixer is attention over shared key/value heads, with three sets of options: (1) interleaved rotation with
banded frequency scaling, u() on the rotated queries and keys, a window that keeps the first positions; (2) no rotation,
keys that are also the values, the same kind of window, one added to the softmax's denominator, a sigmoid gate on every
output channel; (3) biases, rotate-half rotation of the leading channels, a factor per head on the scores, all earlier
positions. Feed-forwards: a cubic of normed powers between two matrices, or a few of many silu units a token, chosen by
softmax scores plus a correction among the best groups of neighbours, some standing for the input itself, beside one unit
that every token uses.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Sequence

import numpy as np


def unit_rms(x: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------- rotation
def frequencies(rot: dict) -> np.ndarray:
    """[dims / 2] radians a position. With `scaling` (factor, low, high, original): a wavelength below original / high stays,
    one above original / low is divided in frequency by factor, between them the two are blended linearly in original / wavelength."""
    n = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * np.arange(n // 2) / n)
    sc = rot.get("scaling")
    if not sc:
        return f
    factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = np.empty_like(f)
    for i, fi in enumerate(f):
        wave = 2.0 * math.pi / fi
        if wave < original / high:
            out[i] = fi
        elif wave > original / low:
            out[i] = fi / factor
        else:
            s = (original / wave - low) / (high - low)
            out[i] = (1.0 - s) * fi / factor + s * fi
    return out


def rotate(x: np.ndarray, rot: dict, pairing: str, first_position: int = 0) -> np.ndarray:
    """x [T, heads, d]; the first rot.dims channels of every head turn, the others stay. "interleaved" couples channels 2i and
    2i + 1, "half" couples i and i + dims / 2."""
    n = int(rot["dims"])
    f = frequencies(rot)
    out = x.copy()
    for t in range(x.shape[0]):
        for i in range(n // 2):
            a, b = (2 * i, 2 * i + 1) if pairing == "interleaved" else (i, i + n // 2)
            angle = (first_position + t) * f[i]
            c, s = math.cos(angle), math.sin(angle)
            u, v = x[t, :, a], x[t, :, b]
            out[t, :, a] = u * c - v * s
            out[t, :, b] = v * c + u * s
    return out


# -------------------------------------------------------------------------------- attention
def visible(T: int, mask: Optional[dict]) -> np.ndarray:
    """[T, T] bool: whether query i sees key j."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    see = j <= i
    if mask:
        see = see & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))
    return see


def softmax_attention(q: np.ndarray, k: np.ndarray, v: np.ndarray, scale, see: np.ndarray, plus_one: bool = False) -> np.ndarray:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; head h reads group h // (H / G); `scale` a number or one per head.
    `plus_one`: weights exp(s_j) / (1 + sum exp(s_j))."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    scale = np.broadcast_to(np.asarray(scale, dtype=np.float64), (H,))
    for h in range(H):
        g = h // per
        s = np.where(see, (q[:, h] @ k[:, g].T) * scale[h], -np.inf)
        top = s.max(-1, keepdims=True)
        if plus_one:
            top = np.maximum(top, 0.0)
        a = np.exp(s - top)
        total = a.sum(-1, keepdims=True)
        if plus_one:
            total = total + np.exp(-top)
        out[:, h] = (a / total) @ v[:, g]
    return out


def normed_window_attention(m: dict, w: Dict[str, np.ndarray], p: str, h: np.ndarray, eps: float) -> np.ndarray:
    H, G, d, e, T = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), h.shape[0]
    q = unit_rms(rotate((h @ w[p + "q"].T).reshape(T, H, d), m["rot"], "interleaved"), eps)
    k = unit_rms(rotate((h @ w[p + "k"].T).reshape(T, G, d), m["rot"], "interleaved"), eps)
    v = (h @ w[p + "v"].T).reshape(T, G, e)
    o = softmax_attention(q, k, v, float(m["scale"]), visible(T, m.get("mask")))
    return o.reshape(T, H * e) @ w[p + "o"].T


def shared_value_attention(m: dict, w: Dict[str, np.ndarray], p: str, h: np.ndarray, eps: float) -> np.ndarray:
    H, G, d, T = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), h.shape[0]
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    k = (h @ w[p + "k"].T).reshape(T, G, d)
    o = softmax_attention(q, k, k, float(m["scale"]), visible(T, m.get("mask")), plus_one=True).reshape(T, H * d)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def tempered_attention(m: dict, w: Dict[str, np.ndarray], p: str, h: np.ndarray, eps: float) -> np.ndarray:
    H, G, d, e, T = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), h.shape[0]
    q = rotate((h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, d), m["rot"], "half")
    k = rotate((h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, d), m["rot"], "half")
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, e)
    o = softmax_attention(q, k, v, float(m["scale"]) * w[p + "temp"], visible(T, None))
    return o.reshape(T, H * e) @ w[p + "o"].T


MIXERS = {"attention": normed_window_attention, "attention_2": shared_value_attention, "attention_3": tempered_attention}


# ---------------------------------------------------------------------------- feed-forwards
def poly_norm(z: np.ndarray, act: np.ndarray, eps: float) -> np.ndarray:
    a, b, c, e = (float(x) for x in act)
    return a * unit_rms(z, eps) + b * unit_rms(z * z, eps) + c * unit_rms(z ** 3, eps) + e


def poly_unit(w: Dict[str, np.ndarray], p: str, x: np.ndarray, eps: float) -> np.ndarray:
    return poly_norm(x @ w[p + "up"].T, w[p + "act"], eps) @ w[p + "down"].T


def gated_unit(w: Dict[str, np.ndarray], p: str, x: np.ndarray) -> np.ndarray:
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def choice_scores(z: np.ndarray, correction: np.ndarray):
    s = np.exp(z - z.max(-1, keepdims=True))
    s = s / s.sum(-1, keepdims=True)
    return s, s + correction


def route(z: np.ndarray, correction: np.ndarray, top: int, groups: int = 1, keep: int = 1):
    """z [n] router outputs of one token. Returns (ids, weights, margin): the chosen outputs, their scores over the scores' sum,
    and by how much the choice is decided (the smaller of the gap between the last group kept and the first dropped and the gap
    between the last output chosen and the first left out; infinite where nothing is left out)."""
    s, c = choice_scores(z, correction)
    n = len(z) // groups
    best = np.array([c[g * n:(g + 1) * n].max() for g in range(groups)])
    ranked = np.argsort(-best, kind="stable")
    margin = best[ranked[keep - 1]] - best[ranked[keep]] if keep < groups else np.inf
    open_ = np.full(len(z), -np.inf)
    for g in ranked[:keep]:
        open_[g * n:(g + 1) * n] = c[g * n:(g + 1) * n]
    order = np.argsort(-open_, kind="stable")
    ids = order[:top]
    if top < keep * n:
        margin = min(margin, open_[order[top - 1]] - open_[order[top]])
    return ids, s[ids] / (s[ids].sum() + 1e-20), margin


def routed_units(f: dict, w: Dict[str, np.ndarray], p: str, x: np.ndarray, margins: Optional[list] = None) -> np.ndarray:
    r = f["router"]
    real, top = int(r["experts"]), int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = x @ w[p + "router"].T
    assert z.shape[1] == real + int(r.get("identity", 0))
    y = np.zeros_like(x)
    decided = np.empty(x.shape[0])
    for t in range(x.shape[0]):
        ids, wt, decided[t] = route(z[t], w[p + "correction"], top, int(groups["count"]), int(groups["keep"]))
        for e, c in zip(ids, wt):
            y[t] += c * (x[t] if e >= real else gated_unit(w, p + f"e{e}.", x[t:t + 1])[0])
    if margins is not None:
        margins.append(decided)
    if f.get("shared") is not None:
        y = y + gated_unit(w, p + "shared.", x)
    return y


def feed_forward(f: dict, w: Dict[str, np.ndarray], p: str, x: np.ndarray, eps: float, margins: Optional[list] = None) -> np.ndarray:
    if f["kind"] == "dense":
        return poly_unit(w, p, x, eps)
    if f["kind"] == "moe":
        return routed_units(f, w, p, x, margins)
    raise ValueError(f"unknown feed-forward kind {f['kind']}")


# ---------------------------------------------------------------------------------- model
def token_side(cfg: dict, w: Dict[str, np.ndarray], i: int, tokens: Sequence[int], s: np.ndarray) -> np.ndarray:
    """What the layer's slice of the side table, gated by the stream, adds to it."""
    d = int(cfg["token_side"]["dim"])
    p = f"l{i}.side."
    e = w["side.embed"][np.asarray(tokens, dtype=np.int64)][:, i * d:(i + 1) * d]
    y = (gelu_tanh(s @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return unit_rms(y, float(cfg["norm"]["eps"])) * w[p + "norm"]


def running_order(cfg: dict) -> List[tuple]:
    """[(layer, pass that starts here or None)] in the order in which the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    order = [(i, None) for i in range(a)]
    for t in range(times):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def pass_input(s: np.ndarray, s0: np.ndarray, t: int, step: np.ndarray) -> np.ndarray:
    return (s + s0 if t > 0 else s) + step[t]


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens: Sequence[int], streams: Optional[list] = None,
            margins: Optional[list] = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence from its first token. `streams` (a list) takes the stream after every layer run.
    `margins` (a list) takes, per routed layer run, by how much each token's choice of units is decided."""
    eps, r = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    s0 = w["embed"][np.asarray(tokens, dtype=np.int64)].astype(np.float64)
    s = s0
    for i, t in running_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            s = pass_input(s, s0, t, w["loop.step"])
        h = unit_rms(s, eps) * w[p + "norm1"]
        s = s + r * unit_rms(MIXERS[layer["type"]](layer["mixer"], w, p + "mix.", h, eps), eps) * w[p + "norm1b"]
        if layer.get("mlp") is not None:
            y = feed_forward(layer["mlp"], w, p + "mlp.", unit_rms(s, eps) * w[p + "norm2"], eps, margins)
            s = s + r * unit_rms(y, eps) * w[p + "norm2b"]
        if cfg.get("token_side"):
            s = s + r * token_side(cfg, w, i, tokens, s)
        if streams is not None:
            streams.append(s)
    return (unit_rms(s, eps) * w["final.norm"]) @ w["embed"].T


def router_margins(cfg: dict, w: Dict[str, np.ndarray], tokens: Sequence[int]) -> np.ndarray:
    margins: list = []
    forward(cfg, w, tokens, margins=margins)
    return np.min(np.stack(margins), 0) if margins else np.full(len(tokens), np.inf)
