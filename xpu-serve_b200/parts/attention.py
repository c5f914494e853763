"""Grouped-query attention over the paged cache, with per-head q/k norms, rotary position
encoding and an optional sigmoid gate per head (src/models/common/blocks.cpp:143-187,
src/models/lfm3/lfm3_decoder.cpp:114-141).

One matrix product gives q, k, v and the gate logits: the four weights are stacked at
load ([q; k; v; gate], the gate rows padded to a multiple of 8). The cache keeps normed,
rotated keys and raw values. A call that reads another call's cache computes q (and the
gate) only.

Masks: every earlier key; a sliding window (`window`); or the query's own block of `chunk`
positions, counted from the sequence's first position (the kernels take one number: 0, W or -C).

Value heads of another size than the key heads (`v_dim`). v_layout "padded" (without rotation): q, k
and v heads are laid out in `padded_head_dim(spec)` channels, the surplus rows of their weights (and
columns of the output projection) being zero: scores and outputs do not change. The per-head norms
then see a mean over more channels; their eps and weights are scaled so that the result is the norm
over head_dim. v_layout "own": keys and values each have a size of their own in the kernels and the
cache, padded in the same way to the next size that the tensor-core kernels take.

Options (config/spec.py: AttentionSpec): a window that keeps the sequence's first positions
(`keep_first`; the cache keeps their pages); queries and keys of unit root mean square behind the
rotation (`unit_qk`: a rotation keeps lengths, so the norm is taken in front of it, by the kernel that
norms, with a weight of ones); keys that are the values (`shared_kv`: one vector a position in the cache,
loaded once for both products); one added to the softmax's denominator (`plus_one`); a gate on every
output channel (`out_gate`, in the attention kernels' epilogues); a factor per head on the scores
(`head_temp`, on the queries as they are stored). A rotation of some of a head's channels, or of
neighbouring ones, is brought into the kernels' pairing by the order of the weights' rows (`channel_layout`). Causal filters
over time on q, k and v (`qkv_taps`; their last inputs are part of a sequence's state) and norms over whole projections
(`qk_norm_all`) run with the rotation and the cache write in one kernel (csrc/qkv_filter.cu); a soft cap on the scores
(`softcap`) in the attention kernels; an output bias (`o_bias`) in the output product.
"""
from __future__ import annotations

from dataclasses import replace
from typing import Dict, List, Tuple

import torch

from .. import registry
from ..config.spec import RopeSpec, ScaledRopeSpec
from ..ops import lib as ops
from .base import KVNeed, Mixer, StateNeed, TensorSpec


def decode_splits(tiles: int, blocks: int, slots: int, fixed: float = 2.0) -> int:
    """Into how many parts to cut each sequence's keys when every sequence brings one token: `tiles` CTAs
    (sequences x kv heads) would each walk `blocks` 64-key blocks; `slots` CTAs run at one time. The cost of a
    choice is its number of rounds of CTAs times a CTA's length (its blocks and a fixed cost worth about two),
    plus the combine kernel when there is more than one part, which walks the parts one after another (a third
    of a block each; measured on B200: one sequence of 2,048 keys takes 9 us in 8 parts, 13 us in 32).
    64 sequences of 2,048 keys over 444 slots: one part is 2 rounds of 35, four parts are 5 rounds of 11."""
    best, best_cost = 1, None
    for parts in range(1, max(1, min(blocks, 64)) + 1):
        rounds = -(-tiles * parts // slots)
        cost = rounds * (-(-blocks // parts) + fixed) + (1.5 + parts / 3.0 if parts > 1 else 0.0)
        if best_cost is None or cost < best_cost - 1e-9:
            best, best_cost = parts, cost
    return best


_TENSOR_CORE_HEAD_DIMS = (16, 32, 48, 64, 96, 128)
_TENSOR_CORE_VALUE_DIMS = (32, 64, 128)      # beside keys of another size (csrc/attention_pairs.cu)


def padded_head_dim(spec) -> int:
    """The one head size in which a layer's q, k and v heads are laid out: head_dim, unless the value heads differ (or it is odd);
    then the next size the tensor-core kernels take, or the next even number above 128."""
    vd = spec.v_dim or spec.head_dim
    if vd == spec.head_dim and vd % 2 == 0:
        return spec.head_dim
    m = max(vd, spec.head_dim)
    for d in _TENSOR_CORE_HEAD_DIMS:
        if m <= d:
            return d
    return m + (m & 1)


def head_sizes(spec) -> Tuple[int, int]:
    """(D, DV): the sizes in which query/key heads and value heads are laid out. "padded": one size for both. "own": the next
    sizes that the tensor-core kernels take, or (above 128) the next even number. Both above 32 and at most 64 become 64, the
    size that the tcgen05 kernel of prompts and the TMA-fed kernel of single tokens take (48 and 64, 16 heads over 4, 2,048
    tokens: the mma.sync kernel at 48 / 64 takes longer than the tcgen05 kernel at 64 / 64)."""
    if spec.v_layout != "own":
        D = padded_head_dim(spec)
        return D, D
    hd, vd = spec.head_dim, spec.v_dim or spec.head_dim
    if 32 < hd <= 64 and 32 < vd <= 64:
        return 64, 64
    D = next((d for d in _TENSOR_CORE_HEAD_DIMS if hd <= d), hd + (hd & 1))
    if spec.shared_kv:
        return D, D
    return D, next((d for d in sorted({D, *_TENSOR_CORE_VALUE_DIMS}) if vd <= d), vd + (vd & 1))


def channel_layout(spec, D: int) -> List[int]:
    """For each of the D channels in which the kernels hold a query or key head: which of the checkpoint's head_dim channels
    stands there (-1: none, zero). The kernels rotate channels i and i + D/2 together: the two members of each pair that
    turns go to the same place of the two halves, then the channels that do not turn."""
    hd, pos = spec.head_dim, spec.position
    if pos is None:
        return list(range(hd)) + [-1] * (D - hd)
    dims = pos.dims if isinstance(pos, ScaledRopeSpec) else hd
    inter = getattr(pos, "pairing", "half") == "interleaved"
    first = [2 * i if inter else i for i in range(dims // 2)]
    second = [2 * i + 1 if inter else i + dims // 2 for i in range(dims // 2)]
    if not isinstance(pos, ScaledRopeSpec):
        return first + second                    # (pairs that do not turn have frequency 0 in the table)
    still = list(range(dims, hd))
    room = D // 2 - dims // 2
    a, b = still[:room], still[room:]
    return first + a + [-1] * (room - len(a)) + second + b + [-1] * (room - len(b))


def _arrange_heads(t: torch.Tensor, heads: int, d: int, layout: List[int]) -> torch.Tensor:
    """[heads * d, ...] -> [heads * len(layout), ...]: every head's rows in the layout's order, zeros where it names none."""
    if layout == list(range(d)):
        return t
    t = t.reshape(heads, d, *t.shape[1:])
    t = torch.cat([t, torch.zeros(heads, 1, *t.shape[2:], dtype=t.dtype)], 1)
    at = torch.tensor([c if c >= 0 else d for c in layout])
    return t[:, at].reshape(heads * len(layout), *t.shape[2:])


class AttentionMixer(Mixer):
    kind = "attention"
    fuses_norm = True
    fixed_shape_ok = True
    concat_output = True

    @classmethod
    def tensors(cls, spec) -> Dict[str, TensorSpec]:
        n = spec.names
        vd = spec.v_dim or spec.head_dim
        qd, kd = spec.heads * spec.head_dim, spec.kv_heads * spec.head_dim
        own_v = spec.own_kv and not spec.shared_kv
        out = {n["q"]: TensorSpec((qd, spec.hidden))}
        if spec.own_kv:
            out[n["k"]] = TensorSpec((kd, spec.hidden))
        if own_v:
            out[n["v"]] = TensorSpec((spec.kv_heads * vd, spec.hidden))
        out[n["o"]] = TensorSpec((spec.hidden, spec.heads * vd))
        if spec.head_gate:
            out[n["gate"]] = TensorSpec((spec.heads, spec.hidden))
        if spec.out_gate:
            out[n["gate"]] = TensorSpec((spec.heads * vd, spec.hidden))
        if spec.qk_norm:
            out[n["q_norm"]] = TensorSpec((spec.head_dim,), init="ones", role="vector")
            if spec.own_kv:
                out[n["k_norm"]] = TensorSpec((spec.head_dim,), init="ones", role="vector")
        if spec.qkv_bias:
            out[n["q_bias"]] = TensorSpec((qd,), role="vector")
            if spec.own_kv:
                out[n["k_bias"]] = TensorSpec((kd,), role="vector")
            if own_v:
                out[n["v_bias"]] = TensorSpec((spec.kv_heads * vd,), role="vector")
        if spec.qkv_taps:
            for key, rows in (("q_conv", qd), ("k_conv", kd), ("v_conv", spec.kv_heads * vd)):
                out[n[key]] = TensorSpec((rows, spec.qkv_taps), init="uniform:-0.5:0.5", role="vector")
        if spec.qk_norm_all:
            out[n["q_norm"]] = TensorSpec((qd,), init="ones", role="vector")
            out[n["k_norm"]] = TensorSpec((kd,), init="ones", role="vector")
        if spec.o_bias:
            out[n["o_bias"]] = TensorSpec((spec.hidden,), role="vector")
        if spec.head_temp:
            out[n["temp"]] = TensorSpec((spec.heads,), init="uniform:0.5:1.5", role="vector")
        return out

    @classmethod
    def cache_need(cls, spec):
        # (a block mask keeps every key: a reader of this cache may have another mask)
        D, DV = head_sizes(spec)
        window = spec.window if not spec.chunk else 0
        kv = KVNeed(spec.kv_heads, D, window, planes=1 if spec.shared_kv else 2, keep_first=spec.keep_first if window > 0 else 0,
                    v_dim=DV if DV != D else 0)
        if spec.qkv_taps > 1:
            return kv, StateNeed((spec.qkv_taps - 1, spec.heads * D + spec.kv_heads * (D + DV)), "compute")
        return kv

    def __init__(self, spec, weights: Dict[str, torch.Tensor], rt):
        vd = spec.v_dim or spec.head_dim
        D, DV = self.D, self.DV = head_sizes(spec)
        if D % 2 != 0 or max(D, DV) > 256:
            raise ValueError(f"attention: head sizes {spec.head_dim} / {vd} must be even (or differ) and at most 256")
        if spec.heads % spec.kv_heads != 0:
            raise ValueError(f"attention: {spec.heads} heads over {spec.kv_heads} kv heads")
        if spec.chunk and spec.window:
            raise ValueError("attention: a layer has a window or a block mask, not both")
        if spec.shared_kv and vd != spec.head_dim:
            raise ValueError(f"attention: keys that are the values have one size, not {spec.head_dim} and {vd}")
        if spec.shared_kv and (spec.position is not None or spec.qk_norm or spec.unit_qk):
            raise ValueError("attention: keys that are the values as projected are neither rotated nor normed")
        if D != spec.head_dim and isinstance(spec.position, RopeSpec):
            raise ValueError("attention: value heads of another size than the key heads need a layer without rotation")
        if spec.qk_norm and spec.unit_qk or spec.head_gate and spec.out_gate:
            raise ValueError("attention: a layer has learned or unit q/k norms, a gate per head or per channel, not both")
        if spec.unit_qk and getattr(getattr(spec.position, "scaling", None), "mscale_k", 0.0) != 0.0:
            raise ValueError("attention: unit queries and keys behind a rotation that changes lengths are not supported")
        self.filtered = spec.qkv_taps > 0 or spec.qk_norm_all      # q, k and v pass the kernel of csrc/qkv_filter.cu
        if self.filtered and (not spec.own_kv or spec.shared_kv or spec.qk_norm or spec.unit_qk or spec.head_temp):
            raise ValueError("attention: filters and norms over whole projections need keys and values of the layer's own, no other norm "
                             "and no factor on the scores")
        if not 0 <= spec.qkv_taps <= 16 or not spec.softcap >= 0.0:
            raise ValueError(f"attention: {spec.qkv_taps} taps (at most 16), soft cap {spec.softcap}")
        if not spec.scale > 0.0 or spec.keep_first < 0:
            raise ValueError("attention: the scale must be positive and keep_first not negative")
        self.spec, self.rt = spec, rt
        self.mask = -int(spec.chunk) if spec.chunk else int(spec.window)     # the kernels' one number
        n = spec.names
        self.planes = 1 if spec.shared_kv else 2
        self.q_dim, self.o_dim = spec.heads * D, spec.heads * DV
        self.kv_cols = spec.kv_heads * (D + (DV if self.planes == 2 else 0))
        # what the kernels need beside the window: passed on to each of them
        self.options = dict(keep=int(spec.keep_first) if spec.window > 0 else 0, planes=self.planes, plus_one=bool(spec.plus_one),
                            gate_channels=bool(spec.out_gate), softcap=float(spec.softcap))
        # the per-head norm over head_dim channels, computed over D: sum / D + eps' = (head_dim / D) (sum / head_dim + eps)
        self.qk_eps = float(spec.qk_norm_eps) * spec.head_dim / D
        norm_scale = (spec.head_dim / D) ** 0.5
        # A checkpoint whose rotation couples other channels than i and i + D/2 is brought into that order here, for q and k
        # alike (their products do not change), and the per-head norm weights with them.
        hd = spec.head_dim
        layout = channel_layout(spec, D)
        v_layout = list(range(vd)) + [-1] * (DV - vd)

        def keys(t: torch.Tensor, heads: int) -> torch.Tensor:         # rows (or elements) of q or k, head by head
            return _arrange_heads(t, heads, hd, layout)

        def values(t: torch.Tensor, heads: int) -> torch.Tensor:
            return _arrange_heads(t, heads, vd, v_layout)

        own_v = spec.own_kv and not spec.shared_kv
        wq = keys(weights[n["q"]], spec.heads)
        q_rows = [wq]
        rows = [wq]
        if spec.own_kv:
            rows.append(keys(weights[n["k"]], spec.kv_heads))
        if own_v:
            rows.append(values(weights[n["v"]], spec.kv_heads))
        biases = q_biases = None
        if spec.qkv_bias:
            bq = keys(weights[n["q_bias"]], spec.heads)
            q_biases = [bq]
            biases = [bq]
            if spec.own_kv:
                biases.append(keys(weights[n["k_bias"]], spec.kv_heads))
            if own_v:
                biases.append(values(weights[n["v_bias"]], spec.kv_heads))
        if spec.head_gate or spec.out_gate:
            g = values(weights[n["gate"]], spec.heads) if spec.out_gate else weights[n["gate"]]
            pad = (-g.shape[0]) % 16      # (whole 16-row tiles: what the few-row product's unpredicated instances and its tails ask for)
            if pad:
                g = torch.cat([g, torch.zeros(pad, g.shape[1], dtype=g.dtype)], 0)
            rows.append(g)
            q_rows.append(g)
            if biases is not None:
                biases.append(torch.zeros(g.shape[0]))
                q_biases.append(torch.zeros(g.shape[0]))
        self.w_qkvg = self.b_qkvg = self.w_qg = self.b_qg = None
        if spec.own_kv:
            self.w_qkvg = rt.matrix(torch.cat([r.to(torch.float32) for r in rows], 0))
            self.b_qkvg = rt.vector(torch.cat([b.to(torch.float32) for b in biases])) if biases is not None else None
        self._q_rows, self._q_biases = q_rows, q_biases          # stacked on the device on the first use as a reader of another cache
        w_o = weights[n["o"]]
        if DV != vd:        # zero columns where the padded value channels stand
            w_o = values(w_o.t().contiguous(), spec.heads).t().contiguous()
        self.w_o = rt.matrix(w_o)
        self.b_o = rt.vector(weights[n["o_bias"]]) if spec.o_bias else None

        self.taps = None
        if self.filtered:
            # [taps, channels], row b for the tap that looks b tokens back (one tap of 1 where only the norms are wanted)
            def filters(key, arrange, heads, d):
                if not spec.qkv_taps:
                    return arrange(torch.ones(heads * d, 1), heads)
                return arrange(weights[n[key]].to(torch.float32).reshape(heads * d, spec.qkv_taps), heads)
            self.taps = rt.vector(torch.cat([filters("q_conv", keys, spec.heads, hd), filters("k_conv", keys, spec.kv_heads, hd),
                                             filters("v_conv", values, spec.kv_heads, vd)], 0).flip(1).t())

        def norm_weight(w: torch.Tensor):
            return rt.vector(keys(w.to(torch.float32), 1) * norm_scale)

        self.q_norm = self.k_norm = None
        if spec.qk_norm:
            self.q_norm = norm_weight(weights[n["q_norm"]])
            self.k_norm = norm_weight(weights[n["k_norm"]]) if spec.own_kv else None
        elif spec.qk_norm_all:
            self.q_norm = rt.vector(keys(weights[n["q_norm"]].to(torch.float32), spec.heads))
            self.k_norm = rt.vector(keys(weights[n["k_norm"]].to(torch.float32), spec.kv_heads))
        elif spec.unit_qk:
            self.q_norm = self.k_norm = norm_weight(torch.ones(hd))
        self.q_scale = rt.vector(weights[n["temp"]]) if spec.head_temp else None
        position = spec.position
        if isinstance(position, ScaledRopeSpec):      # (one table entry per pair of the layout)
            position = replace(position, pairs=D // 2)
        self.position = registry.position_class(position.kind)(position, rt) if position is not None else None

    def takes_prenormed(self, rows: int) -> bool:
        return (self.w_qkvg is not None and self.rt.few_rows_shape(rows, self.w_qkvg) and self.w_qkvg.shape[1] % 8 == 0)

    def scale_output(self, s: float) -> bool:
        """What the heads leave is linear in the values, and those in their filters, which are float32."""
        if self.taps is None:
            return s == 1.0
        self.taps[:, self.q_dim + self.spec.kv_heads * self.D:] *= s
        return True

    def forward(self, x, step, cache, into=None) -> torch.Tensor:
        T = x.shape[0]
        o = self.rt.ws.get("attn_o", (T, self.o_dim), self.rt.act_dtype)
        self.heads(x, step, cache, o)
        if into is not None:
            return into.product(o, self.w_o, self.b_o)
        return self.rt.linear(o, self.w_o, "mixer_out", self.b_o)

    def heads(self, x, step, cache, out) -> None:
        """Everything in front of the output projection, into `out` [tokens, o_dim] (columns of any matrix)."""
        s, rt = self.spec, self.rt
        T = x.shape[0]
        if cache is None or cache.storage is None:
            raise RuntimeError("attention needs a key/value cache")
        D, DV = self.D, self.DV
        if cache.owner:
            if self.w_qkvg is None:
                raise RuntimeError("attention: a layer without keys and values of its own must read another call's cache")
            w_in, b_in, gate_at = self.w_qkvg, self.b_qkvg, self.q_dim + self.kv_cols
        else:
            if self.w_qg is None:
                self.w_qg = rt.matrix(torch.cat([r.to(torch.float32) for r in self._q_rows], 0))
                if self._q_biases is not None:
                    self.b_qg = rt.vector(torch.cat([b.to(torch.float32) for b in self._q_biases]))
            w_in, b_in, gate_at = self.w_qg, self.b_qg, self.q_dim
        table = step.page_tables[cache.group]
        rope = self.position.table(step.max_positions) if self.position is not None else None
        q = rt.ws.get("attn_q", (T, s.heads, D), rt.act_dtype)
        if self.filtered:
            if not cache.owner or len(cache) != (2 if s.qkv_taps > 1 else 1):
                raise RuntimeError("attention with filtered projections keeps its own keys, values and filter inputs")
            # (the filter's kernel adds the biases: a filter starts from zeros, not from biases)
            proj = rt.linear(x, w_in, "attn_qkv")
            ops.qkv_filter(proj, b_in, self.taps, cache[1].storage if s.qkv_taps > 1 else None, q, cache[0].storage, table,
                           step.seq_of_token, step.positions, step.cu_seqlens, step.slots, self.q_norm, self.k_norm, rope, s.heads,
                           s.kv_heads, D, DV, step.page_size, s.qk_norm_eps, s.heads * s.head_dim, s.kv_heads * s.head_dim,
                           all_single=step.decode)
        elif step.decode and D == DV and self.planes == 2 and self.q_scale is None and rt.rope_behind_product(x, w_in, D):
            # one token a sequence: the per-head norms, the rotation and the cache write run behind the product, in its kernel
            proj = rt.ws.get("attn_qkv", (T, w_in.shape[0]), rt.act_dtype)
            rt.few_rows_rope(x, w_in, proj, b_in, q_out=q, pool=cache.storage if cache.owner else None,
                             page_table=table if cache.owner else None, seq_of_token=step.seq_of_token,
                             positions=step.positions, q_w=self.q_norm, k_w=self.k_norm, rope=rope, heads=s.heads,
                             kv_heads=s.kv_heads, head_dim=D, page_size=step.page_size, eps=self.qk_eps)
        else:
            # (the vendor's product has no float32 bias: with many rows the kernel behind it adds the biases)
            late = b_in if b_in is not None and rt.mode == "bfloat16" and rt.many_rows == "auto" and not rt.few_rows(x, w_in) else None
            proj = rt.linear(x, w_in, "attn_qkv", None if late is not None else b_in)
            ops.qk_norm_rope_store(proj, q, cache.storage, table, step.seq_of_token, step.positions, self.q_norm,
                                   self.k_norm, rope, s.heads, s.kv_heads, D, step.page_size, self.qk_eps,
                                   write_kv=cache.owner, v_dim=DV, planes=self.planes, q_scale=self.q_scale, bias=late)
        gate = proj[:, gate_at:] if s.head_gate or s.out_gate else None
        self.attend(q, cache, table, step, gate, out.unflatten(1, (s.heads, DV)))

    def attend(self, q, cache, table, step, gate, o) -> None:
        s, rt, D, DV, mask = self.spec, self.rt, self.D, self.DV, self.mask
        group = s.heads // s.kv_heads
        mma = rt.mode == "bfloat16" and ops.attention_mma_supports(D, step.page_size, group, DV)
        tc = mma and rt.prompt_attention == "tcgen05" and D == DV and ops.attention_tc_supports(D, step.page_size, group)
        if step.fixed_shape and mma:
            # a step captured for any lengths up to its bounds: one key split, grids from the bounds
            if tc:
                ops.attention_tc(q, cache.storage, table, step.cu_seqlens, step.kv_lens, gate, o, step.n_seqs,
                                 step.max_q_len, s.kv_heads, step.page_size, s.scale, mask, step.max_kv_len, **self.options)
            else:
                ops.attention_mma(q, cache.storage, table, step.cu_seqlens, step.kv_lens, gate, o, None, step.n_seqs,
                                  step.max_q_len, s.kv_heads, step.page_size, s.scale, mask, 1, **self.options)
            return
        if mma:
            # Few tiles and long key ranges (decoding): split each range over several CTAs so that
            # every SM streams a part of the cache; the partial results meet in scratch memory.
            tokens_per_tile = 64 // group
            tiles = sum(-(-int(n) // tokens_per_tile) for n in step.q_lens_host) * s.kv_heads
            blocks = -(-step.max_kv_len // step.page_size)
            if s.window > 0 or s.chunk > 0:       # the keys a tile can see span at most so many pages
                blocks = min(blocks, -(-(max(s.window, s.chunk) + step.max_q_len) // step.page_size) + 1
                             + -(-self.options["keep"] // step.page_size))
            if step.decode and group <= 16 and rt.attn_split_factor == 0:
                splits = decode_splits(tiles, blocks, max(1, ops.attention_mma_decode_slots(D, tiles, DV, self.planes)),
                                       rt.attn_fixed_cost)
            else:
                splits = max(1, min(blocks, 32, (max(rt.attn_split_factor, 1) * rt.sm_count) // max(tiles, 1)))
            # prompts: the tcgen05 kernel, unless few tiles face many keys (a short piece of a long sequence), where
            # cutting the keys over more CTAs is worth more
            if tc and (splits == 1 or step.max_kv_len <= 512) and not step.decode:
                ops.attention_tc(q, cache.storage, table, step.cu_seqlens, step.kv_lens, gate, o, step.n_seqs,
                                 step.max_q_len, s.kv_heads, step.page_size, s.scale, mask, step.max_kv_len, **self.options)
                return
            scratch = None
            if splits > 1:
                need = ops.attention_mma_scratch_bytes(q.shape[0] * s.heads, DV, splits)
                scratch = rt.ws.get("attn_scratch", (need,), torch.uint8)
            counters = rt.attn_counters if (rt.fuse_tails and rt.tail_attn and step.n_seqs * s.kv_heads <= rt.attn_counters.numel()) else None
            ops.attention_mma(q, cache.storage, table, step.cu_seqlens, step.kv_lens, gate, o, scratch, step.n_seqs,
                              step.max_q_len, s.kv_heads, step.page_size, s.scale, mask, splits, counters=counters,
                              bounded_waits=step.decode, **self.options)
            return
        ops.attention_generic(q, cache.storage, table, step.seq_of_token, step.positions, gate, o, s.kv_heads,
                              step.page_size, s.scale, mask, **self.options)


registry.register_mixer(AttentionMixer.kind, AttentionMixer)
