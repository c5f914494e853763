"""Typed configuration of Lazovik, read from config.json's own keys.

config.json gives the model's `width`, `vocab`, `norm.eps`, `loop` (`start`, `stop`, `times`: layers start .. stop - 1 run `times`
times in a row with the same weights, each pass with a cache and state of its own, behind a learned vector per pass; absent:
every layer once) and under `layers` one entry per layer: `type` (which mixer), `mixer` (its sizes and constants) and `mlp` (its
feed-forward, or null for none). Every size and every constant that can differ between two models of the design is read from
there, but for how many hidden entries a decay's low-rank matrices have: the checkpoint's tensors decide that (`rank` in a
mixer's entry says what a model with random weights gets).

Layer types:
  parallel   `left`: attention (`heads`, `kv_heads`, `dim`, `vdim`) over blocks of `mask.size` positions, biases, filters of
             `conv` taps on q, k and v, norms over whole projections, rotate-half rotation of the first `rot.dims` channels
             (`rot.base`, `rot.scaling`: factor, original, fast, slow), scores times `scale` under a cap (`softcap`), a
             sigmoid gate per channel; beside `right`: time mixing (`heads` of `dim`); summed times `left_scale`, `right_scale`
  gla        gated linear attention (`heads`, `dim`, `vdim`, `tau`)
Feed-forward (`mlp.kind` "moe"): `router.experts` squared-ReLU units of `expert.ff`, of which a token uses `router.top`, chosen
by sigmoid scores and fed the score times the token; `shared.ff`: a unit every token uses, behind a sigmoid gate.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .json_util import ConfigError, get_float, get_float_or, get_int, get_int_or, get_str
from .spec import (AttentionSpec, GatedLinearSpec, LayerCall, LayerSpec, ModelSpec, NormSpec, RopeScalingSpec, RoutedExpertsSpec,
                   ScaledRopeSpec, SquaredReluSpec, SummedMixerSpec, TimeMixingSpec)

PARALLEL, GLA = "parallel", "gla"
MAX_POSITION = 1 << 20               # the design has no table of positions; this only bounds what a cache is sized for
RANDOM_RANK = 16                     # of a decay's low-rank matrices, in a model with random weights that names none

_LAYER_NAMES = {"pre_mixer": "norm1", "pre_ffn": "norm2"}
_LEFT_NAMES = {"q": "mix.left.q", "k": "mix.left.k", "v": "mix.left.v", "o": "mix.left.o", "gate": "mix.left.g",
               "q_norm": "mix.left.q.norm", "k_norm": "mix.left.k.norm", "q_bias": "mix.left.q.b", "k_bias": "mix.left.k.b",
               "v_bias": "mix.left.v.b", "o_bias": "mix.left.o.b", "q_conv": "mix.left.q.conv", "k_conv": "mix.left.k.conv",
               "v_conv": "mix.left.v.conv"}
_RIGHT_NAMES = {**{f"mu_{s}": f"mix.right.mu.{s}" for s in "rkvgw"}, **{s: f"mix.right.{s}" for s in ("r", "k", "v", "w1", "w2", "w0", "u", "norm", "o")},
                "gate": "mix.right.g"}


def _obj(d: dict, key: str, where: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: missing object '{key}'")
    return v


def _rank(m: dict, where: str) -> int:
    rank = get_int_or(m, "rank", RANDOM_RANK, where)
    if rank <= 0:
        raise ConfigError(f"{where}: rank must be positive")
    return rank


@dataclass(frozen=True)
class LazovikLayer:
    type: str
    mixer: object                    # SummedMixerSpec | GatedLinearSpec
    mlp: Optional[RoutedExpertsSpec]
    raw: dict                        # the entry as read (written back by to_json)


@dataclass(frozen=True)
class LazovikConfig:
    vocab: int
    width: int
    norm_eps: float
    loop: Optional[Tuple[int, int, int]]     # (start, stop, times)
    layers: Tuple[LazovikLayer, ...]
    architecture: str = "Lazovik"

    # ---------------------------------------------------------------- parsing
    @staticmethod
    def _rotation(m: dict, dim: int, where: str) -> ScaledRopeSpec:
        rot = _obj(m, "rot", where)
        base, dims = get_float(rot, "base", f"{where} rot"), get_int(rot, "dims", f"{where} rot")
        if not base > 0 or base == 1.0 or dims <= 0 or dims % 2 != 0 or dims > dim:
            raise ConfigError(f"{where} rot: base must be positive (and not 1) and dims even, positive and at most dim")
        scaling = None
        if rot.get("scaling") is not None:
            sw = f"{where} rot.scaling"
            sc = _obj(rot, "scaling", f"{where} rot")
            scaling = RopeScalingSpec(factor=get_float(sc, "factor", sw), original=get_float(sc, "original", sw),
                                      fast=get_float(sc, "fast", sw), slow=get_float(sc, "slow", sw))
            if not min(scaling.factor, scaling.original, scaling.fast, scaling.slow) > 0:
                raise ConfigError(f"{sw}: factor, original, fast and slow must be positive")
        return ScaledRopeSpec(head_dim=dim, theta=base, dims=dims, scaling=scaling)

    @classmethod
    def _left(cls, m: dict, width: int, eps: float, where: str) -> AttentionSpec:
        heads, kv_heads = get_int(m, "heads", where), get_int(m, "kv_heads", where)
        dim, vdim = get_int(m, "dim", where), get_int(m, "vdim", where)
        scale, softcap = get_float(m, "scale", where), get_float_or(m, "softcap", 0.0, where)
        taps = get_int_or(m, "conv", 0, where)
        if min(heads, kv_heads, dim, vdim) <= 0 or heads % kv_heads != 0 or not scale > 0:
            raise ConfigError(f"{where}: heads, kv_heads, dim, vdim and scale must be positive and kv_heads divide heads")
        if not 0 <= taps <= 16 or softcap < 0:
            raise ConfigError(f"{where}: conv must be at most 16 taps and softcap not negative")
        chunk = 0
        if m.get("mask") is not None:
            chunk = get_int(_obj(m, "mask", where), "size", f"{where} mask")
            if chunk <= 0:
                raise ConfigError(f"{where} mask: size must be positive")
        return AttentionSpec(hidden=width, heads=heads, kv_heads=kv_heads, head_dim=dim, v_dim=vdim, v_layout="own", qk_norm=False,
                             qk_norm_all=True, qk_norm_eps=eps, position=cls._rotation(m, dim, where), window=0, chunk=chunk,
                             head_gate=False, out_gate=True, scale=scale, softcap=softcap, qkv_bias=True, o_bias=True, qkv_taps=taps,
                             names=dict(_LEFT_NAMES))

    @staticmethod
    def _right(m: dict, width: int, eps: float, where: str) -> TimeMixingSpec:
        heads, dim = get_int(m, "heads", where), get_int(m, "dim", where)
        if min(heads, dim) <= 0:
            raise ConfigError(f"{where}: heads and dim must be positive")
        return TimeMixingSpec(hidden=width, heads=heads, dim=dim, rank=_rank(m, where), eps=eps, names=dict(_RIGHT_NAMES))

    @classmethod
    def _mixer(cls, kind: str, m: dict, width: int, eps: float, where: str):
        if kind == PARALLEL:
            scales = (get_float(m, "left_scale", where), get_float(m, "right_scale", where))
            return SummedMixerSpec(hidden=width, scales=scales, branches=(cls._left(_obj(m, "left", where), width, eps, f"{where} left"),
                                                                         cls._right(_obj(m, "right", where), width, eps, f"{where} right")))
        if kind == GLA:
            heads, dim, vdim = get_int(m, "heads", where), get_int(m, "dim", where), get_int(m, "vdim", where)
            tau = get_float(m, "tau", where)
            if min(heads, dim, vdim) <= 0 or not tau > 0:
                raise ConfigError(f"{where}: heads, dim, vdim and tau must be positive")
            return GatedLinearSpec(hidden=width, heads=heads, dim=dim, vdim=vdim, rank=_rank(m, where), tau=tau, eps=eps)
        raise ConfigError(f"{where}: unknown layer type '{kind}' ({PARALLEL}, {GLA})")

    @staticmethod
    def _mlp(f: Optional[dict], width: int, where: str) -> Optional[RoutedExpertsSpec]:
        if f is None:
            return None
        if not isinstance(f, dict):
            raise ConfigError(f"{where}: 'mlp' must be an object or null")
        kind = get_str(f, "kind", where)
        if kind != "moe":
            raise ConfigError(f"{where}: unknown feed-forward kind '{kind}' (moe)")
        router = _obj(f, "router", where)
        experts, top = get_int(router, "experts", f"{where} router"), get_int(router, "top", f"{where} router")
        ff = get_int(_obj(f, "expert", where), "ff", f"{where} expert")
        if ff <= 0 or experts <= 0 or not 0 < top <= experts:
            raise ConfigError(f"{where}: expert.ff, router.experts and router.top must be positive and top at most experts")
        shared = None
        if f.get("shared") is not None:
            sff = get_int(_obj(f, "shared", where), "ff", f"{where} shared")
            if sff <= 0:
                raise ConfigError(f"{where} shared: ff must be positive")
            shared = SquaredReluSpec(hidden=width, intermediate=sff, names={"up": "mlp.shared.up", "down": "mlp.shared.down"})
        return RoutedExpertsSpec(hidden=width, intermediate=ff, experts=experts, top=top, score="sigmoid", activation="relu_squared",
                                 weight_on="input", shared=shared)

    @classmethod
    def from_json(cls, cfg: dict) -> "LazovikConfig":
        w = "config.json"
        width, vocab = get_int(cfg, "width", w), get_int(cfg, "vocab", w)
        eps = get_float(_obj(cfg, "norm", w), "eps", f"{w} norm")
        if min(width, vocab) <= 0 or not eps > 0:
            raise ConfigError(f"{w}: width, vocab and norm.eps must be positive")
        entries = cfg.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError(f"{w}: 'layers' must be a list with at least one entry")
        layers = []
        for i, e in enumerate(entries):
            where = f"{w} layers[{i}]"
            if not isinstance(e, dict):
                raise ConfigError(f"{where}: must be an object")
            kind = get_str(e, "type", where)
            mixer = cls._mixer(kind, _obj(e, "mixer", where), width, eps, f"{where} mixer")
            layers.append(LazovikLayer(kind, mixer, cls._mlp(e.get("mlp"), width, f"{where} mlp"), e))
        loop = None
        if cfg.get("loop") is not None:
            lp = _obj(cfg, "loop", w)
            loop = (get_int(lp, "start", f"{w} loop"), get_int(lp, "stop", f"{w} loop"), get_int(lp, "times", f"{w} loop"))
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ConfigError(f"{w} loop: needs 0 <= start < stop <= {len(layers)} layers and times >= 1")
        return cls(vocab=vocab, width=width, norm_eps=eps, loop=loop, layers=tuple(layers))

    def to_json(self) -> dict:
        out = {"architecture": self.architecture, "layers": [l.raw for l in self.layers], "norm": {"eps": self.norm_eps},
               "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return out

    # ------------------------------------------------------- to a model spec
    def running_order(self) -> Tuple[LayerCall, ...]:
        n = len(self.layers)
        if self.loop is None:
            return tuple(LayerCall(i) for i in range(n))
        a, b, times = self.loop
        calls = [LayerCall(i) for i in range(a)]
        for t in range(times):
            calls += [LayerCall(i, step_row=t if i == a else None) for i in range(a, b)]
        return tuple(calls + [LayerCall(i) for i in range(b, n)])

    def model_spec(self) -> ModelSpec:
        norm = NormSpec(self.width, self.norm_eps)
        layers = tuple(LayerSpec(prefix=f"l{i}.", mixer=l.mixer, ffn=l.mlp, norm=norm, sandwich=False, kind="pre_norm", names=dict(_LAYER_NAMES))
                       for i, l in enumerate(self.layers))
        spec = ModelSpec(arch="lazovik", vocab=self.vocab, hidden=self.width, max_position=MAX_POSITION, layers=layers,
                         order=self.running_order(), final_norm=norm, tied_head=False, init_std=0.05, prefixes=("",),
                         # a layer without a feed-forward may still carry the norm of one
                         ignorable=tuple(rf"^l{i}\.norm2$" for i, l in enumerate(self.layers) if l.mlp is None),
                         pass_steps=self.loop[2] if self.loop is not None else 0,
                         names={"embed": "embed", "final_norm": "final.norm", "head": "head", "pass_step": "loop.step"})
        spec.validate()
        return spec
