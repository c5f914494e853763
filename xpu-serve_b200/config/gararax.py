"""Typed configuration of Gararax, read from config.json's own keys.

config.json gives the model's `width`, `vocab`, `norm.eps`, `residual_mult` (a constant on every branch, behind its norm),
`token_side.dim` (channels of the second token table that every layer reads; absent: no such input), `loop` (`start`,
`stop`, `times`: layers start .. stop - 1 run `times` times in a row with the same weights, each pass with a cache of its
own, behind a learned vector per pass and, from the second on, the embedding's output; absent: every layer once) and under
`layers` one entry per layer: `type` (which mixer), `mixer` (its sizes and constants) and `mlp` (its feed-forward, or null
for none). Every size and every constant that can differ between two models of the design is read from there.

Layer types, all attention (`heads`, `kv_heads`, `dim`, `vdim`, `scale`):
  attention     interleaved rotation (`rot.base`, `rot.dims`, `rot.scaling`: factor, low, high, original), queries and keys of
                unit root mean square, a sliding window that keeps the first positions (`mask.size`, `mask.keep_first`)
  attention_2   no rotation, keys that are the values, the same kind of window, one added to the softmax's denominator, a
                sigmoid gate on every output channel
  attention_3   biases on q, k and v, rotate-half rotation of the first `rot.dims` channels, a learned factor per head on
                the scores, every earlier position
Feed-forwards (`mlp.kind`): `dense` (PolyNorm between two matrices of `ff`), `moe` (`router.experts` silu units of
`expert.ff`, of which a token uses `router.top`, chosen by softmax scores plus a correction among the best `groups.keep` of
`groups.count` groups and weighted by the scores over their sum; the last `router.identity` router outputs stand for the
token's input itself; `shared.ff`: a unit every token uses).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .json_util import ConfigError, get_float, get_int, get_int_or, get_str
from .spec import (AttentionSpec, BandRopeScalingSpec, LayerCall, LayerSpec, ModelSpec, NormSpec, PolyNormSpec,
                   RoutedExpertsSpec, ScaledRopeSpec, SwiGLUSpec, TokenSideSpec)

NORMED, SHARED_VALUES, TEMPERED = "attention", "attention_2", "attention_3"
MAX_POSITION = 1 << 20               # the design has no table of positions; this only bounds what a cache is sized for

_LAYER_NAMES = {"pre_mixer": "norm1", "post_mixer": "norm1b", "pre_ffn": "norm2", "post_ffn": "norm2b"}
_MIXER_NAMES = {"q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o", "gate": "mix.g", "temp": "mix.temp",
                "q_bias": "mix.q.b", "k_bias": "mix.k.b", "v_bias": "mix.v.b"}


def _obj(d: dict, key: str, where: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: missing object '{key}'")
    return v


@dataclass(frozen=True)
class GararaxLayer:
    type: str
    mixer: AttentionSpec
    mlp: Optional[object]            # PolyNormSpec | RoutedExpertsSpec | None
    raw: dict                        # the entry as read (written back by to_json)


@dataclass(frozen=True)
class GararaxConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    side_dim: int                    # 0: no per-layer token input
    loop: Optional[Tuple[int, int, int]]     # (start, stop, times)
    layers: Tuple[GararaxLayer, ...]
    architecture: str = "Gararax"

    # ---------------------------------------------------------------- parsing
    @staticmethod
    def _rotation(m: dict, dim: int, pairing: str, where: str) -> ScaledRopeSpec:
        rot = _obj(m, "rot", where)
        base, dims = get_float(rot, "base", f"{where} rot"), get_int(rot, "dims", f"{where} rot")
        if not base > 0 or dims <= 0 or dims % 2 != 0 or dims > dim:
            raise ConfigError(f"{where} rot: base must be positive and dims even, positive and at most dim")
        scaling = None
        if rot.get("scaling") is not None:
            sw = f"{where} rot.scaling"
            sc = _obj(rot, "scaling", f"{where} rot")
            scaling = BandRopeScalingSpec(factor=get_float(sc, "factor", sw), low=get_float(sc, "low", sw),
                                          high=get_float(sc, "high", sw), original=get_float(sc, "original", sw))
            if not (scaling.factor > 0 and scaling.original > 0 and scaling.high > scaling.low):
                raise ConfigError(f"{sw}: factor and original must be positive and high above low")
        return ScaledRopeSpec(head_dim=dim, theta=base, dims=dims, scaling=scaling, pairing=pairing)

    @staticmethod
    def _mask(m: dict, where: str) -> Tuple[int, int]:
        """(window, first positions kept)"""
        if m.get("mask") is None:
            return 0, 0
        mask = _obj(m, "mask", where)
        size, keep = get_int(mask, "size", f"{where} mask"), get_int_or(mask, "keep_first", 0, f"{where} mask")
        if size <= 0 or keep < 0:
            raise ConfigError(f"{where} mask: size must be positive and keep_first not negative")
        return size, keep

    @classmethod
    def _mixer(cls, kind: str, m: dict, width: int, eps: float, where: str) -> AttentionSpec:
        heads, kv_heads = get_int(m, "heads", where), get_int(m, "kv_heads", where)
        dim, vdim = get_int(m, "dim", where), get_int(m, "vdim", where)
        scale = get_float(m, "scale", where)
        if min(heads, kv_heads, dim, vdim) <= 0 or heads % kv_heads != 0 or not scale > 0:
            raise ConfigError(f"{where}: heads, kv_heads, dim, vdim and scale must be positive and kv_heads divide heads")
        common = dict(hidden=width, heads=heads, kv_heads=kv_heads, head_dim=dim, v_dim=vdim, v_layout="own", qk_norm=False,
                      qk_norm_eps=eps, head_gate=False, scale=scale, names=dict(_MIXER_NAMES))
        if kind == NORMED:
            window, keep = cls._mask(m, where)
            return AttentionSpec(position=cls._rotation(m, dim, "interleaved", where), window=window, keep_first=keep, unit_qk=True,
                                 **common)
        if kind == SHARED_VALUES:
            if vdim != dim:
                raise ConfigError(f"{where}: the values are the keys, so vdim must equal dim")
            window, keep = cls._mask(m, where)
            return AttentionSpec(position=None, window=window, keep_first=keep, shared_kv=True, plus_one=True, out_gate=True, **common)
        if kind == TEMPERED:
            return AttentionSpec(position=cls._rotation(m, dim, "half", where), window=0, qkv_bias=True, head_temp=True, **common)
        raise ConfigError(f"{where}: unknown layer type '{kind}' ({NORMED}, {SHARED_VALUES}, {TEMPERED})")

    @staticmethod
    def _mlp(f: Optional[dict], width: int, eps: float, where: str):
        if f is None:
            return None
        if not isinstance(f, dict):
            raise ConfigError(f"{where}: 'mlp' must be an object or null")
        kind = get_str(f, "kind", where)
        if kind == "dense":
            ff = get_int(f, "ff", where)
            if ff <= 0:
                raise ConfigError(f"{where}: ff must be positive")
            return PolyNormSpec(hidden=width, intermediate=ff, eps=eps)
        if kind != "moe":
            raise ConfigError(f"{where}: unknown feed-forward kind '{kind}' (dense, moe)")
        router, expert = _obj(f, "router", where), _obj(f, "expert", where)
        rw = f"{where} router"
        experts, top, identity = get_int(router, "experts", rw), get_int(router, "top", rw), get_int_or(router, "identity", 0, rw)
        count = keep = 1
        if router.get("groups") is not None:
            groups = _obj(router, "groups", rw)
            count, keep = get_int(groups, "count", f"{rw} groups"), get_int(groups, "keep", f"{rw} groups")
        ff = get_int(expert, "ff", f"{where} expert")
        outputs = experts + identity
        if ff <= 0 or experts <= 0 or identity < 0 or top <= 0:
            raise ConfigError(f"{where}: expert.ff, router.experts and router.top must be positive, router.identity not negative")
        if count <= 0 or outputs % count != 0 or not 0 < keep <= count or top > keep * (outputs // count):
            raise ConfigError(f"{where}: groups.count must divide the router's {outputs} outputs, and the groups.keep groups that "
                              f"stay open hold at least router.top of them")
        shared = None
        if f.get("shared") is not None:
            sff = get_int(_obj(f, "shared", where), "ff", f"{where} shared")
            if sff <= 0:
                raise ConfigError(f"{where} shared: ff must be positive")
            shared = SwiGLUSpec(hidden=width, intermediate=sff, activation="silu",
                                names={"gate": "mlp.shared.gate", "up": "mlp.shared.up", "down": "mlp.shared.down"})
        return RoutedExpertsSpec(hidden=width, intermediate=ff, experts=experts, top=top, score="softmax_all", correction=True,
                                 identity=identity, groups=count, keep_groups=keep, group_top=1, renorm=True, renorm_eps=1e-20,
                                 shared=shared, shared_gated=False)

    @classmethod
    def from_json(cls, cfg: dict) -> "GararaxConfig":
        w = "config.json"
        width, vocab = get_int(cfg, "width", w), get_int(cfg, "vocab", w)
        eps = get_float(_obj(cfg, "norm", w), "eps", f"{w} norm")
        mult = get_float(cfg, "residual_mult", w)
        if min(width, vocab) <= 0 or not eps > 0:
            raise ConfigError(f"{w}: width, vocab and norm.eps must be positive")
        side_dim = 0
        if cfg.get("token_side") is not None:
            side_dim = get_int(_obj(cfg, "token_side", w), "dim", f"{w} token_side")
            if side_dim <= 0:
                raise ConfigError(f"{w} token_side: dim must be positive")
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
            layers.append(GararaxLayer(kind, mixer, cls._mlp(e.get("mlp"), width, eps, f"{where} mlp"), e))
        loop = None
        if cfg.get("loop") is not None:
            lp = _obj(cfg, "loop", w)
            loop = (get_int(lp, "start", f"{w} loop"), get_int(lp, "stop", f"{w} loop"), get_int(lp, "times", f"{w} loop"))
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ConfigError(f"{w} loop: needs 0 <= start < stop <= {len(layers)} layers and times >= 1")
        return cls(vocab=vocab, width=width, norm_eps=eps, residual_mult=mult, side_dim=side_dim, loop=loop, layers=tuple(layers))

    def to_json(self) -> dict:
        out = {"architecture": self.architecture, "layers": [l.raw for l in self.layers], "norm": {"eps": self.norm_eps},
               "residual_mult": self.residual_mult, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        return out

    # ------------------------------------------------------- to a model spec
    def running_order(self) -> Tuple[LayerCall, ...]:
        n = len(self.layers)
        if self.loop is None:
            return tuple(LayerCall(i) for i in range(n))
        a, b, times = self.loop
        calls = [LayerCall(i) for i in range(a)]
        for t in range(times):
            calls += [LayerCall(i, step_row=t if i == a else None, add_embedding=(i == a and t > 0)) for i in range(a, b)]
        return tuple(calls + [LayerCall(i) for i in range(b, n)])

    def model_spec(self) -> ModelSpec:
        norm = NormSpec(self.width, self.norm_eps)
        n = len(self.layers)
        layers = tuple(
            LayerSpec(prefix=f"l{i}.", mixer=l.mixer, ffn=l.mlp, norm=norm, sandwich=True, kind="pre_norm",
                      names=dict(_LAYER_NAMES), branch_scale=self.residual_mult,
                      token_side=(TokenSideSpec(dim=self.side_dim, offset=i * self.side_dim, columns=n * self.side_dim,
                                                vocab=self.vocab, eps=self.norm_eps, scale=self.residual_mult)
                                  if self.side_dim else None))
            for i, l in enumerate(self.layers))
        spec = ModelSpec(arch="gararax", vocab=self.vocab, hidden=self.width, max_position=MAX_POSITION, layers=layers,
                         order=self.running_order(), final_norm=norm, tied_head=True, init_std=0.05, prefixes=("",),
                         # a layer without a feed-forward may still carry the norms of one
                         ignorable=tuple(rf"^l{i}\.norm2b?$" for i, l in enumerate(self.layers) if l.mlp is None),
                         pass_steps=self.loop[2] if self.loop is not None else 0,
                         names={"embed": "embed", "final_norm": "final.norm", "head": "head", "pass_step": "loop.step"})
        spec.validate()
        return spec
