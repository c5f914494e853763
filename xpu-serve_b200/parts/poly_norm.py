"""PolyNorm feed-forward: down(act(up y)), act(z) = a N(z) + b N(z^2) + c N(z^3) + e with N a division by the root mean
square over the token's intermediate values and (a, b, c, e) four learned numbers. One product, one kernel over its rows
(csrc/poly_norm.cu: three sums of powers and the cubic, float32), one product."""
from __future__ import annotations

from typing import Dict

import torch

from .. import registry
from ..ops import lib as ops
from .base import FeedForward, TensorSpec


class PolyNormUnit(FeedForward):
    kind = "poly_norm"
    fixed_shape_ok = True

    @classmethod
    def tensors(cls, spec) -> Dict[str, TensorSpec]:
        n = spec.names
        return {n["up"]: TensorSpec((spec.intermediate, spec.hidden)), n["down"]: TensorSpec((spec.hidden, spec.intermediate)),
                n["act"]: TensorSpec((4,), init="uniform:-1:1", role="vector")}

    def __init__(self, spec, weights: Dict[str, torch.Tensor], rt):
        self.spec, self.rt = spec, rt
        n = spec.names
        self.w_up, self.w_down = rt.matrix(weights[n["up"]]), rt.matrix(weights[n["down"]])
        self.coef = rt.vector(weights[n["act"]])

    def forward(self, y, step) -> torch.Tensor:
        rt, s = self.rt, self.spec
        z = rt.linear(y, self.w_up, "ffn_up")
        act = rt.ws.get("ffn_act", (y.shape[0], s.intermediate), rt.act_dtype)
        ops.poly_norm(z, self.coef, act, s.eps)
        return rt.linear(act, self.w_down, "ffn_out")


registry.register_ffn(PolyNormUnit.kind, PolyNormUnit)
