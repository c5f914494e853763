"""Tiny Lazovik configurations for the tests, and helpers to write them as model folders with random weights.

A has sizes that are no multiple of 8 and differ from layer to layer: value heads larger and smaller than key heads, filters of
two to five taps, blocks of 13 and 29 positions, decays through 5 and 11 hidden entries, rotations of some channels with and
without frequency scaling, top 2 of 6 and top 3 of 5, a layer without a feed-forward, one without a shared unit, a loop over
the two middle layers that runs three times. B has sizes that the tensor-core kernels take (keys of 64 with values of 64, of 128
with values of 32, memories of 64 x 128 and 128 x 64), blocks longer and shorter than a page, one query head a key head, a loop
that starts at the first layer. C has no loop, blocks of one position and of exactly a page, filters of one tap, one head, every
expert chosen. D has no experts (so that every place can be compared in bfloat16, where a router's close calls cut B's
comparisons short). The single-layer configurations run each mechanism alone; `whole_loop` repeats every layer.
"""
import os

from xpu_serve_b200.config import LazovikConfig
from xpu_serve_b200.weights import write_random_model


def rotation(dims, base, scaling=None):
    rot = {"dims": dims, "base": float(base)}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return rot


def left(heads, kv_heads, dim, vdim, size, rot, conv=3, scale=0.3, softcap=4.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": size}, "rot": rot,
            "scale": scale, "softcap": softcap}


def right(heads, dim, rank=6):
    return {"heads": heads, "dim": dim, "rank": rank}


def parallel(l, r, left_scale=0.8, right_scale=1.3):
    return "parallel", {"left": l, "right": r, "left_scale": left_scale, "right_scale": right_scale}


def gla(heads, dim, vdim, tau, rank=7):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}


def moe(ff, experts, top, shared_ff=0):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared_ff:
        f["shared"] = {"ff": shared_ff}
    return f


def model(width, vocab, layers, loop=None, eps=1e-5):
    cfg = {"architecture": "Lazovik", "width": width, "vocab": vocab, "norm": {"eps": eps},
           "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


SCALING = (3.0, 64, 8.0, 1.0)

CONFIGS = {
    "A": model(44, 203, [
        (parallel(left(6, 3, 12, 20, 13, rotation(6, 100.0, SCALING), conv=2), right(3, 10, rank=5)), moe(20, 6, 2, 12)),
        (gla(3, 10, 14, 3.0, rank=11), moe(12, 5, 3)),
        (parallel(left(4, 1, 14, 6, 29, rotation(14, 500.0), conv=5, scale=0.5, softcap=2.5), right(2, 6), -0.6, 0.7), None),
        (gla(2, 18, 5, 9.0), moe(16, 3, 1, 20)),
    ], loop=(1, 3, 3), eps=3e-6),
    "B": model(128, 384, [
        (parallel(left(8, 2, 64, 64, 70, rotation(32, 10000.0, (8.0, 128, 4.0, 0.5)), conv=4, scale=0.2), right(4, 64, rank=24)), moe(48, 8, 3, 64)),
        (gla(2, 64, 128, 8.0, rank=16), moe(64, 4, 2, 32)),
        (parallel(left(4, 4, 128, 32, 150, rotation(64, 3000.0), conv=3, scale=0.1, softcap=9.0), right(8, 16, rank=8), 1.1, 0.4), None),
        (gla(4, 128, 64, 16.0, rank=40), moe(40, 16, 4, 64)),
    ], loop=(0, 2, 2), eps=0.2),
    "C": model(64, 180, [
        (parallel(left(2, 2, 32, 48, 64, rotation(16, 200.0), conv=1), right(1, 24)), moe(24, 2, 2, 16)),
        (gla(1, 40, 8, 1.0), None),
        (parallel(left(1, 1, 16, 16, 1, rotation(2, 50.0), conv=2), right(5, 8), 0.5, 0.5), moe(8, 3, 3)),
    ]),
    "D": model(96, 250, [
        (parallel(left(10, 2, 64, 64, 90, rotation(64, 500.0, (4.0, 200, 16.0, 1.0)), conv=3, scale=0.125, softcap=20.0), right(2, 48, rank=16)), None),
        (gla(6, 32, 64, 5.0, rank=12), None),
        (parallel(left(6, 3, 48, 64, 64, rotation(16, 3000.0), conv=2, scale=0.2), right(4, 32)), None),
        (gla(2, 96, 32, 16.0), None),
    ], loop=(1, 4, 2), eps=0.2),
    # one mechanism's neighbourhood each
    "parallel": model(40, 150, [(parallel(left(4, 2, 10, 6, 9, rotation(6, 50.0, (2.0, 40, 4.0, 1.0))), right(2, 12)), None)]),
    "memory": model(40, 150, [(gla(3, 12, 20, 4.0), None)]),
    "routed": model(40, 150, [(gla(1, 8, 8, 2.0), moe(30, 7, 3, 20))]),
    "whole_loop": model(48, 150, [(parallel(left(2, 1, 16, 32, 30, rotation(8, 100.0)), right(2, 16)), None), (gla(2, 16, 16, 6.0), None)],
                        loop=(0, 2, 3)),
    # sizes that only the generic kernels take, memories beyond 128 key channels and with values in several blocks
    "wide_heads": model(48, 150, [(parallel(left(2, 1, 160, 72, 50, rotation(80, 500.0), scale=0.08), right(1, 136)), None),
                                  (gla(2, 200, 40, 7.0), None), (gla(1, 24, 300, 7.0), None)]),
}

# What makes a lost part show: routers, gates, decays, the bonus, biases, pass vectors and the token table at a size that matters.
SCALE = {".mlp.router": 2.5, ".mlp.shared.sg": 4.0, ".up": 2.0, ".down": 1.5, ".left.g": 4.0, ".right.g": 3.0, ".mix.g": 3.0, "embed": 10.0, "loop.step": 12.0,
         ".b": 6.0, ".w1": 3.0, ".w2": 4.0, ".a1": 2.0, ".a2": 6.0, ".left.q.norm": 2.0, ".left.k.norm": 1.5}


# B and D have a large eps and seeds of their own: a head's output is divided by its root mean square, and with a small eps a
# token whose read nearly cancels turns the whole head around with a rounding of bfloat16.
SEEDS = {"B": 41, "D": 38}


def make_folder(root, name: str, dtype: str, seed: int = 0, std: float = 0.08):
    seed = seed or SEEDS.get(name, 37)
    folder = os.path.join(str(root), f"lazovik_{name}_{dtype}")
    if not os.path.isdir(folder):
        write_random_model(folder, LazovikConfig.from_json(CONFIGS[name]), seed=seed, dtype=dtype, std=std,
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
    """Largest |difference| / largest |reference logit| that rounding alone may cause: float32 5e-6 a layer run, at least 1e-5
    (memories that add up hundreds of tokens, and norms that divide a head's output by its root mean square); bfloat16 about ten roundings to 8 bits a layer run that add like a random walk, times 3 for the largest of many logits."""
    runs = layer_runs(name)
    return max(1e-5, 5e-6 * runs) if dtype == "float32" else 3.0 * (10.0 * runs) ** 0.5 * U_BF16
