"""Mixers side by side: every branch reads the same input. ParallelMixer's result is

    scale * sum_k  out_k / sqrt(mean(out_k^2) + eps) * w_k

each branch's output normed over the model's width with a weight of its own before the sum (float32). A branch is any
registered mixer; what the branches keep per sequence stands one behind another in the call's declaration, and each
branch is handed the view of its own part. SummedMixer's is sum_k scale_k out_k, with no norm between: the branches leave
their output projections to it (parts/base.py: `concat_output`), their heads stand side by side in one matrix, and one
product with the projections side by side gives the sum (in decode steps it adds it to the stream itself).
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import registry
from ..ops import lib as ops
from .base import Mixer, TensorSpec


def _needs_of(need) -> tuple:
    return () if need is None else tuple(need) if isinstance(need, (tuple, list)) else (need,)


class ParallelMixer(Mixer):
    kind = "parallel"
    fixed_shape_ok = True      # (its branches must be too: checked when they are built)

    @classmethod
    def tensors(cls, spec) -> Dict[str, TensorSpec]:
        out: Dict[str, TensorSpec] = {}
        for branch in spec.branches:
            out.update(registry.mixer_class(branch.kind).tensors(branch))
        for name in spec.out_names:
            out[name] = TensorSpec((spec.hidden,), init="ones", role="vector")
        return out

    @classmethod
    def cache_need(cls, spec):
        needs = ()
        for branch in spec.branches:
            needs += _needs_of(registry.mixer_class(branch.kind).cache_need(branch))
        return needs if needs else None

    def __init__(self, spec, weights: Dict[str, torch.Tensor], rt):
        if not spec.branches or len(spec.branches) != len(spec.out_names):
            raise ValueError("parallel mixer: one output weight per branch, and at least one branch")
        self.spec, self.rt = spec, rt
        self.branches = [registry.mixer_class(b.kind)(b, weights, rt) for b in spec.branches]
        self.out_w = [rt.vector(weights[name]) for name in spec.out_names]
        self.spans = []
        at = 0
        for b in spec.branches:
            n = len(_needs_of(registry.mixer_class(b.kind).cache_need(b)))
            self.spans.append((at, at + n))
            at += n
        if not all(getattr(m, "fixed_shape_ok", False) for m in self.branches):
            raise ValueError("parallel mixer: every branch's prompt code must be capturable for any lengths (fixed_shape_ok)")

    def forward(self, x, step, cache) -> torch.Tensor:
        s, rt = self.spec, self.rt
        acc = rt.ws.get("parallel_sum", (x.shape[0], s.hidden), torch.float32)
        for k, (mixer, w, (lo, hi)) in enumerate(zip(self.branches, self.out_w, self.spans)):
            y = mixer.forward(x, step, cache.sub(lo, hi) if cache is not None else None)
            ops.rmsnorm_accumulate(y, w, acc, s.eps, s.scale, add=k > 0)
        return acc


class SummedMixer(Mixer):
    kind = "parallel_sum"
    fuses_norm = True          # (its input is read by products and by other kernels: the normed tensor; its output product adds to the stream)
    fixed_shape_ok = True

    @classmethod
    def tensors(cls, spec) -> Dict[str, TensorSpec]:
        out: Dict[str, TensorSpec] = {}
        for branch in spec.branches:
            out.update(registry.mixer_class(branch.kind).tensors(branch))
        return out

    @classmethod
    def cache_need(cls, spec):
        return ParallelMixer.cache_need(spec)

    def __init__(self, spec, weights: Dict[str, torch.Tensor], rt):
        if not spec.branches or len(spec.branches) != len(spec.scales):
            raise ValueError("summed mixers: one scale per branch, and at least one branch")
        self.spec, self.rt = spec, rt
        self.branches = [registry.mixer_class(b.kind)(b, weights, rt) for b in spec.branches]
        if not all(m.concat_output and getattr(m, "fixed_shape_ok", False) for m in self.branches):
            raise ValueError("summed mixers: every branch must leave its output projection to the sum (concat_output) and be capturable "
                             "for any lengths (fixed_shape_ok)")
        self.spans, self.columns = [], []
        at = col = 0
        w, bias = [], None
        for b, m, s in zip(spec.branches, self.branches, spec.scales):
            n = len(_needs_of(registry.mixer_class(b.kind).cache_need(b)))
            self.spans.append((at, at + n))
            at += n
            pad = (-m.o_dim) % 16                  # (whole 16-column pieces: every branch's rows start aligned)
            self.columns.append((col, col + m.o_dim))
            col += m.o_dim + pad
            scaled = m.scale_output(float(s))      # where the branch cannot scale its heads in float32, its matrix is scaled
            w.append(m.w_o if scaled else (m.w_o.float() * float(s)).to(m.w_o.dtype))
            if pad:
                w.append(torch.zeros((spec.hidden, pad), dtype=m.w_o.dtype, device=rt.device))
            if m.b_o is not None:
                bias = m.b_o * float(s) if bias is None else bias + m.b_o * float(s)
            m.w_o = m.b_o = None                   # (held once, in the product below)
        self.width = col
        self.w_o = torch.cat(w, 1).contiguous()
        self.b_o = bias.contiguous() if bias is not None else None

    def forward(self, x, step, cache, into=None) -> Optional[torch.Tensor]:
        rt = self.rt
        T = x.shape[0]
        side = rt.ws.get("summed_heads", (T, self.width), rt.act_dtype)
        for m, (lo, hi), (c0, c1) in zip(self.branches, self.spans, self.columns):
            m.heads(x, step, cache.sub(lo, hi) if cache is not None else None, side[:, c0:c1])
        for (_, c1), nxt in zip(self.columns, [c[0] for c in self.columns[1:]] + [self.width]):
            if nxt > c1:
                side[:, c1:nxt].zero_()            # columns that belong to no head: their weights are zero, what stands there must be finite
        if into is not None:
            return into.product(side, self.w_o, self.b_o)
        return rt.linear(side, self.w_o, "mixer_out", self.b_o)


registry.register_mixer(ParallelMixer.kind, ParallelMixer)
registry.register_mixer(SummedMixer.kind, SummedMixer)
