"""A plain, slow Lazovik in float64 numpy: whole sequences, no cache, one function per mechanism.

It shares no code with the package: it reads config.json's keys itself and takes tensors by their checkpoint names.
Notation: T tokens, W the model's width; rows of a [T, n] array are tokens. Weights are [out, in], applied as y = x M^T;
u(x) = x / sqrt(mean x^2 + eps). The stream starts as rows of the token table, and a layer is

    s = s + mixer(u(s) w1)
    s = s + units(u(s) w2)                                  (layers with a feed-forward)

A span of layers may run several times in a row with the same weights; pass t (from 0 on) starts from s + step[t]. Mixers:
a linear-attention memory with a learned decay per key channel ("gla"); or two side by side ("parallel"): softmax attention
over the query's own block of positions (filters over time on q, k and v, norms over whole projections, a rotation of the
leading channels, capped scores, a gate per channel) beside a memory whose inputs mix neighbouring tokens, with a decay per
key channel and a bonus for the current token. Feed-forwards: squared-ReLU units chosen by sigmoid scores, each fed its score
times the input, beside one that every token uses.
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


# -------------------------------------------------------------------------- inputs over time
def causal_filter(x: np.ndarray, taps: np.ndarray) -> np.ndarray:
    """y[t, c] = sum_b taps[c, n - 1 - b] x[t - b, c], zeros before the first token; taps [channels, n]."""
    n = taps.shape[1]
    y = np.zeros_like(x)
    for b in range(min(n, x.shape[0])):
        y[b:] += x[:x.shape[0] - b] * taps[:, n - 1 - b]
    return y


def previous_token(h: np.ndarray) -> np.ndarray:
    """Row t is h[t - 1], zeros for the first token."""
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]], 0)


def mix_tokens(h: np.ndarray, mu: np.ndarray) -> np.ndarray:
    return h + (previous_token(h) - h) * mu


# -------------------------------------------------------------------------------- rotation
def frequencies(rot: dict):
    """([dims / 2] radians a position, the factor on cosine and sine). With `scaling` (factor, original, fast, slow): pairs that
    turn more than `fast` times over `original` positions keep their frequency, those that turn fewer than `slow` times are
    divided by `factor`, with a linear ramp over the pair's index between."""
    n, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original, fast, slow = (float(sc[k]) for k in ("factor", "original", "fast", "slow"))

    def index_that_turns(t):
        return n * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index_that_turns(fast)), 0), min(math.ceil(index_that_turns(slow)), n - 1)
    out = []
    for i in range(n // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / factor * ramp + f[i] * (1.0 - ramp))
    return np.array(out), 0.1 * math.log(factor) + 1.0


def rotate(x: np.ndarray, rot: dict) -> np.ndarray:
    """x [T, heads, d]; the first rot.dims channels of every head turn, i with i + dims / 2; the others stay."""
    n = int(rot["dims"])
    f, mult = frequencies(rot)
    out = x.copy()
    for t in range(x.shape[0]):
        for i in range(n // 2):
            c, s = math.cos(t * f[i]) * mult, math.sin(t * f[i]) * mult
            a, b = x[t, :, i], x[t, :, i + n // 2]
            out[t, :, i] = a * c - b * s
            out[t, :, i + n // 2] = b * c + a * s
    return out


# -------------------------------------------------------------------------------- attention
def visible(T: int, mask: Optional[dict]) -> np.ndarray:
    """[T, T] bool: whether query i sees key j: the earlier positions of its own block of mask.size positions."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    see = j <= i
    if mask:
        see = see & (i // int(mask["size"]) == j // int(mask["size"]))
    return see


def cap_scores(s: np.ndarray, cap: float) -> np.ndarray:
    return cap * np.tanh(s / cap)


def softmax_attention(q: np.ndarray, k: np.ndarray, v: np.ndarray, scale: float, see: np.ndarray, cap: float = 0.0) -> np.ndarray:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; head h reads group h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if cap:
            s = cap_scores(s, cap)
        s = np.where(see, s, -np.inf)
        a = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (a / a.sum(-1, keepdims=True)) @ v[:, h // per]
    return out


def whole_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    """One norm over all heads of a projection together."""
    return unit_rms(x, eps) * w


def block_attention(m: dict, w: Dict[str, np.ndarray], p: str, h: np.ndarray, eps: float) -> np.ndarray:
    H, G, d, e, T = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), h.shape[0]
    q, k, v = (causal_filter(h @ w[p + n].T + w[p + n + ".b"], w[p + n + ".conv"]) for n in "qkv")
    q = rotate(whole_norm(q, w[p + "q.norm"], eps).reshape(T, H, d), m["rot"])
    k = rotate(whole_norm(k, w[p + "k.norm"], eps).reshape(T, G, d), m["rot"])
    o = softmax_attention(q, k, v.reshape(T, G, e), float(m["scale"]), visible(T, m["mask"]), float(m["softcap"])).reshape(T, H * e)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T + w[p + "o.b"]


# --------------------------------------------------------------------------------- memories
def memory_with_bonus(r, k, v, decay, bonus):
    """r, k, decay [T, H, d], v [T, H, e], bonus [H, d]: a token reads the memory before its own write, plus its own pair with
    the bonus on every key channel."""
    T, H, d = r.shape
    S = np.zeros((H, d, v.shape[2]))
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hde,hd->he", S + bonus[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return o


def memory(q, k, v, decay):
    """A token reads the memory behind its own write."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]))
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hde,hd->he", S, q[t])
    return o


def double_exponential_decay(mix: np.ndarray, w1: np.ndarray, w2: np.ndarray, w0: np.ndarray) -> np.ndarray:
    return np.exp(-np.exp(np.tanh(mix @ w1.T) @ w2.T + w0))


def rooted_sigmoid_decay(h: np.ndarray, a1: np.ndarray, a2: np.ndarray, bias: np.ndarray, tau: float) -> np.ndarray:
    return sigmoid((h @ a1.T) @ a2.T + bias) ** (1.0 / tau)


def time_mixing(m: dict, w: Dict[str, np.ndarray], p: str, h: np.ndarray, eps: float) -> np.ndarray:
    H, d, T = int(m["heads"]), int(m["dim"]), h.shape[0]
    r, k, v, g = (mix_tokens(h, w[p + "mu." + n]) @ w[p + n].T for n in "rkvg")
    decay = double_exponential_decay(mix_tokens(h, w[p + "mu.w"]), w[p + "w1"], w[p + "w2"], w[p + "w0"])
    o = memory_with_bonus(*(x.reshape(T, H, d) for x in (r, k, v, decay)), w[p + "u"])
    return (unit_rms(o, eps).reshape(T, H * d) * w[p + "norm"] * silu(g)) @ w[p + "o"].T


def decayed_attention(m: dict, w: Dict[str, np.ndarray], p: str, h: np.ndarray, eps: float) -> np.ndarray:
    H, d, e, T = int(m["heads"]), int(m["dim"]), int(m["vdim"]), h.shape[0]
    q = (h @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, e)
    decay = rooted_sigmoid_decay(h, w[p + "a1"], w[p + "a2"], w[p + "a2.b"], float(m["tau"])).reshape(T, H, d)
    o = unit_rms(memory(q, k, v, decay), eps) * w[p + "norm"]
    return (o.reshape(T, H * e) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(m: dict, w: Dict[str, np.ndarray], p: str, h: np.ndarray, eps: float) -> np.ndarray:
    return (float(m["left_scale"]) * block_attention(m["left"], w, p + "left.", h, eps)
            + float(m["right_scale"]) * time_mixing(m["right"], w, p + "right.", h, eps))


MIXERS = {"parallel": side_by_side, "gla": decayed_attention}


# ---------------------------------------------------------------------------- feed-forwards
def squared_relu_unit(w: Dict[str, np.ndarray], p: str, x: np.ndarray) -> np.ndarray:
    return np.maximum(x @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def route(z: np.ndarray, top: int):
    """z [n] router outputs of one token -> (chosen units, their scores, by how much the choice is decided)."""
    s = sigmoid(z)
    order = np.argsort(-s, kind="stable")
    margin = s[order[top - 1]] - s[order[top]] if top < len(z) else np.inf
    return order[:top], s[order[:top]], margin


def weighted_unit(w: Dict[str, np.ndarray], p: str, x: np.ndarray, c: float) -> np.ndarray:
    """The weight is on the unit's input."""
    return squared_relu_unit(w, p, c * x)


def routed_units(f: dict, w: Dict[str, np.ndarray], p: str, x: np.ndarray, margins: Optional[list] = None) -> np.ndarray:
    top = int(f["router"]["top"])
    z = x @ w[p + "router"].T
    assert z.shape[1] == int(f["router"]["experts"])
    y = np.zeros_like(x)
    decided = np.empty(x.shape[0])
    for t in range(x.shape[0]):
        ids, weights, decided[t] = route(z[t], top)
        for e, c in zip(ids, weights):
            y[t] += weighted_unit(w, p + f"e{e}.", x[t:t + 1], c)[0]
    if margins is not None:
        margins.append(decided)
    if f.get("shared") is not None:
        y = y + squared_relu_unit(w, p + "shared.", x) * sigmoid(x @ w[p + "shared.sg"].T)
    return y


# ---------------------------------------------------------------------------------- model
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


def pass_input(s: np.ndarray, t: int, step: np.ndarray) -> np.ndarray:
    return s + step[t]


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens: Sequence[int], streams: Optional[list] = None,
            margins: Optional[list] = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence from its first token. `streams` (a list) takes the stream after every layer run.
    `margins` (a list) takes, per routed layer run, by how much each token's choice of units is decided."""
    eps = float(cfg["norm"]["eps"])
    s = w["embed"][np.asarray(tokens, dtype=np.int64)].astype(np.float64)
    for i, t in running_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            s = pass_input(s, t, w["loop.step"])
        s = s + MIXERS[layer["type"]](layer["mixer"], w, p + "mix.", unit_rms(s, eps) * w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            s = s + routed_units(layer["mlp"], w, p + "mlp.", unit_rms(s, eps) * w[p + "norm2"], margins)
        if streams is not None:
            streams.append(s)
    return (unit_rms(s, eps) * w["final.norm"]) @ w["head"].T


def router_margins(cfg: dict, w: Dict[str, np.ndarray], tokens: Sequence[int]) -> np.ndarray:
    margins: list = []
    forward(cfg, w, tokens, margins=margins)
    return np.min(np.stack(margins), 0) if margins else np.full(len(tokens), np.inf)
