"""Tiny Gararax configurations for the tests, and helpers to write them as model folders with random weights.

A has sizes that are no multiple of 8 and differ from layer to layer: value heads larger and smaller than key heads, an odd
head size, a partial rotation, windows of 13 to 21 positions that keep five, nine or no first positions, a layer without a
feed-forward, groups of router outputs that mix experts and pass-through outputs, a loop over the two middle layers that
runs twice. B has sizes that the tensor-core kernels take (keys of 128 with values of 32, keys of 96 with values of 64, equal
heads of 64), more kept positions than the window is long, one group of outputs, top 1, a loop over one layer that runs three
times, a residual factor of 1. C has no loop and no side table, a window of one position, a window that ends at a page's
border and keeps exactly a page, one head, groups of which all stay open. D has no experts (so that every place can be compared
in bfloat16, where a router's close calls cut B's comparisons short) and all three mixers at sizes that the tensor-core kernels
take. The single-layer configurations run each mechanism
alone; `whole_loop` repeats every layer.
"""
import os

from xpu_serve_b200.config import GararaxConfig
from xpu_serve_b200.weights import write_random_model


def rotation(dims, base, scaling=None):
    rot = {"dims": dims, "base": float(base)}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return rot


def normed(heads, kv_heads, dim, vdim, scale, rot, size, keep):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot,
                         "mask": {"size": size, "keep_first": keep}}


def shared(heads, kv_heads, dim, scale, size, keep):
    return "attention_2", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                           "mask": {"size": size, "keep_first": keep}}


def tempered(heads, kv_heads, dim, vdim, scale, rot):
    return "attention_3", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, identity, top, groups=None, shared_ff=0):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}
    if groups:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared_ff:
        f["shared"] = {"ff": shared_ff}
    return f


def model(width, vocab, layers, loop=None, side=0, eps=1e-5, mult=0.7):
    cfg = {"architecture": "Gararax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
           "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


SCALING = (3.0, 1.0, 4.0, 64)

CONFIGS = {
    "A": model(44, 203, [
        (normed(6, 3, 12, 20, 0.31, rotation(12, 100.0, SCALING), 21, 5), dense(50)),
        (shared(4, 1, 10, 0.4, 13, 9), moe(20, 5, 1, 2, (2, 1), 12)),
        (tempered(4, 2, 14, 6, 0.27, rotation(8, 500.0)), None),
        (shared(3, 3, 7, 0.5, 17, 0), moe(12, 4, 2, 3, (3, 2))),
    ], loop=(1, 3, 2), side=5, eps=3e-6),
    "B": model(128, 384, [
        (tempered(8, 2, 128, 32, 0.09, rotation(96, 10000.0)), dense(256)),
        (normed(4, 4, 64, 64, 0.2, rotation(32, 1000.0, (8.0, 0.5, 2.0, 128)), 70, 3), moe(48, 8, 0, 1, None, 64)),
        (shared(6, 2, 64, 0.125, 40, 66), moe(64, 6, 2, 4, (4, 3))),
        (normed(2, 1, 96, 64, 0.1, rotation(96, 200.0), 33, 1), dense(64)),
    ], loop=(1, 2, 3), side=8, mult=1.0),
    "C": model(64, 180, [
        (shared(4, 4, 16, 0.3, 1, 0), dense(40)),
        (normed(4, 2, 32, 16, 0.25, rotation(16, 10000.0), 65, 64), moe(24, 4, 2, 2, (3, 3), 16)),
        (tempered(1, 1, 16, 16, 0.2, rotation(16, 10000.0)), None),
    ], mult=0.25),
    "D": model(96, 250, [
        (shared(10, 2, 64, 0.125, 150, 70), dense(120)),
        (tempered(6, 2, 96, 32, 0.1, rotation(64, 3000.0)), dense(96)),
        (normed(8, 4, 32, 64, 0.3, rotation(32, 500.0, (4.0, 1.0, 4.0, 200)), 90, 11), None),
        (normed(3, 1, 64, 64, 0.15, rotation(16, 500.0), 64, 64), dense(64)),
    ], loop=(0, 3, 2), side=16, mult=0.6),
    # one mechanism's neighbourhood each
    "normed": model(40, 150, [(normed(4, 2, 10, 6, 0.5, rotation(6, 50.0, (2.0, 1.0, 3.0, 40)), 12, 4), None)], side=3),
    "shared_values": model(40, 150, [(shared(4, 2, 12, 0.4, 9, 3), None)]),
    "tempered": model(40, 150, [(tempered(4, 1, 8, 24, 0.4, rotation(4, 50.0)), None)]),
    "poly": model(40, 150, [(shared(1, 1, 8, 0.3, 4, 0), dense(72))]),
    "routed": model(40, 150, [(shared(1, 1, 8, 0.3, 4, 0), moe(30, 7, 2, 3, (3, 2), 20))]),
    "whole_loop": model(48, 150, [(tempered(2, 1, 16, 32, 0.3, rotation(8, 100.0)), dense(32)),
                                  (shared(2, 2, 16, 0.3, 30, 2), None)], loop=(0, 2, 3), side=4),
    # sizes that only the generic kernels take
    "wide_heads": model(48, 150, [(normed(2, 1, 160, 72, 0.08, rotation(80, 500.0), 50, 7), dense(30)),
                                  (tempered(2, 2, 40, 136, 0.2, rotation(24, 500.0)), None)]),
}

# What makes a lost part show: routers, gates, the token tables, the pass vectors, biases and queries at a size that matters.
SCALE = {".mlp.router": 3.0, ".mlp.correction": 3.0, ".mix.g": 4.0, "embed": 10.0, "side.embed": 0.6, ".side.gate": 0.3, "loop.step": 12.0, ".b": 6.0,
         ".mix.q": 2.0, ".mix.k": 2.0, "final.norm": 0.1}


def make_folder(root, name: str, dtype: str, seed: int = 31, std: float = 0.08):
    folder = os.path.join(str(root), f"gararax_{name}_{dtype}")
    if not os.path.isdir(folder):
        write_random_model(folder, GararaxConfig.from_json(CONFIGS[name]), seed=seed, dtype=dtype, std=std,
                           norm_range=(0.5, 1.5), scale=SCALE)
    return folder


def prompt(name: str, length: int, salt: int = 0):
    V = CONFIGS[name]["vocab"]
    return [(i * 31 + 5 + 17 * salt + (i * i) % 13) % V for i in range(length)]


U_BF16 = 2.0 ** -9


def layer_runs(name: str) -> int:
    cfg = CONFIGS[name]
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    return n if not lp else n + (lp["stop"] - lp["start"]) * (lp["times"] - 1)


def upper_limit(name: str, dtype: str) -> float:
    """Largest |difference| / largest |reference logit| that rounding alone may cause: float32 2e-6 a layer run, at least 1e-5
    (every branch ends in a norm over a freshly projected vector); bfloat16 about ten roundings to 8 bits a layer run that add
    like a random walk, times 2 for the largest of many logits."""
    runs = layer_runs(name)
    return max(1e-5, 2e-6 * runs) if dtype == "float32" else 2.0 * (10.0 * runs) ** 0.5 * U_BF16
