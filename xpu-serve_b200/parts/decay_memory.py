"""Two mixers around a memory whose rows (key channels) decay each at a learned rate: S [dim, vdim] per head, float32 and zero at a
sequence's start (csrc/decay_scan.cu).

GatedLinearMixer ("gla"; gated linear attention), input x:

    q = Wq x dim^(-1/2),  k = Wk x  (heads of dim),  v = Wv x  (heads of vdim)
    a = sigmoid(A2 (A1 x) + b)^(1 / tau)                           one per key channel
    S <- diag(a) S + k v^T;   o = S^T q                            (the read sees the token's own write)

then every head's o divided by its root mean square, times a weight of vdim entries that the heads share, times silu(Wg x),
and the output projection.

TimeMixingMixer ("time_mixing"; RWKV-style), with x' the sequence's input before x (zeros for the first) and
m_s = x + (x' - x) mu_s:

    r = Wr m_r,  k = Wk m_k,  v = Wv m_v  (heads of dim),   a = exp(-exp(W2 tanh(W1 m_w) + w0))
    o = (S + diag(u) k v^T)^T r;   S <- diag(a) S + k v^T           (the read comes before the write, the bonus u stands in for it)

then every head's o divided by its root mean square, times a weight over all heads, times silu(Wg m_g), and the projection.

The projections are in the activation type. A1 x and W1 m_w leave their products as float32, and everything behind them (tanh,
the second matrix, the exponentials, the memory and its sums, the heads' norm) is float32 in both precision modes. How many
hidden entries a decay has is the checkpoint's business (TensorSpec.free). Single tokens and short pieces walk in order; long
pieces of a prompt run chunk by chunk side by side.
"""
from __future__ import annotations

import os
from typing import Dict, Optional

import torch

from .. import registry
from ..ops import lib as ops
from .base import Mixer, StateNeed, TensorSpec
from .mamba2 import chunk_plan


class DecayMemoryMixer(Mixer):
    """What the two share: the scan over the memory, chunked or in order, with the heads' norm and gate behind it."""
    fuses_norm = True
    fixed_shape_ok = True      # the kernels find every sequence's tokens in the step's description on the device
    concat_output = True

    def _setup(self, spec, rt, vdim: int, w_norm: torch.Tensor, w_o: torch.Tensor) -> None:
        if spec.dim > 256:
            raise ValueError(f"{spec.kind}: key size {spec.dim} (at most 256 is supported)")
        self.spec, self.rt, self.vdim = spec, rt, vdim
        self.o_dim = spec.heads * vdim
        self.w_norm = rt.vector(w_norm)
        self.w_o = rt.matrix(w_o)
        self.b_o = None
        self.finishes = ops.decay_scan_finishes(spec.dim, vdim)
        # Pieces of at least two chunks run chunk by chunk side by side. XS_DECAY_CHUNK: tokens a chunk (0: always in order);
        # unset: as many chunks as fill the device once, between 32 and 256 tokens each.
        self.chunk = int(os.environ["XS_DECAY_CHUNK"]) if "XS_DECAY_CHUNK" in os.environ else None

    def scale_output(self, s: float) -> bool:
        self.w_norm = self.w_norm * s
        return True

    def forward(self, x, step, cache, into=None) -> Optional[torch.Tensor]:
        rt = self.rt
        out = rt.ws.get("memory_heads", (x.shape[0], self.o_dim), rt.act_dtype)
        self.heads(x, step, cache, out)
        if into is not None:
            return into.product(out, self.w_o)
        return rt.linear(out, self.w_o, "mixer_out")

    def heads(self, x, step, cache, out) -> None:
        raise NotImplementedError

    def _scan(self, q, k, v, decay, state, gate, out, step, q_scale: float, bonus=None) -> None:
        s, rt = self.spec, self.rt
        T = q.shape[0]
        chunk, chunks = self.chunk, None
        if chunk is None:
            at_once = max(1, (ops.decay_scan_ctas(s.dim, self.vdim) * rt.sm_count) // ops.decay_scan_blocks(s.heads, s.dim, self.vdim))
            chunk = min(256, max(32, -(-T // at_once // 8) * 8))
        if chunk > 0 and not step.fixed_shape and not step.decode and step.max_q_len >= 2 * chunk:
            chunk_seq, first_chunk = chunk_plan(step, chunk, rt.device)
            n = chunk_seq.shape[0]
            chunks = (chunk_seq, first_chunk, rt.ws.get("memory_chunk_state", (n, s.heads, s.dim, self.vdim), torch.float32),
                      rt.ws.get("memory_chunk_decay", (n, s.heads, s.dim), torch.float32))
        common = dict(q_scale=q_scale, bonus=bonus, chunks=chunks)
        if self.finishes:
            ops.decay_scan(q, k, v, decay, state, step.cu_seqlens, step.slots, s.heads, s.dim, self.vdim, out=out, norm_w=self.w_norm,
                           gate=gate, eps=s.eps, **common)
            return
        y = rt.ws.get("memory_y", (T, self.o_dim), torch.float32)
        ops.decay_scan(q, k, v, decay, state, step.cu_seqlens, step.slots, s.heads, s.dim, self.vdim, y=y, **common)
        ops.grouped_rmsnorm(y, self.w_norm, out, s.heads, s.eps, gate=gate, gate_act="silu")


class GatedLinearMixer(DecayMemoryMixer):
    kind = "gla"

    @classmethod
    def tensors(cls, spec) -> Dict[str, TensorSpec]:
        n = spec.names
        qd, vd = spec.heads * spec.dim, spec.heads * spec.vdim
        return {
            n["q"]: TensorSpec((qd, spec.hidden)), n["k"]: TensorSpec((qd, spec.hidden)), n["v"]: TensorSpec((vd, spec.hidden)),
            n["gate"]: TensorSpec((vd, spec.hidden)), n["o"]: TensorSpec((spec.hidden, vd)),
            n["norm"]: TensorSpec((spec.vdim,), init="ones", role="vector"),
            n["a1"]: TensorSpec((spec.rank, spec.hidden), free=((0, "a1"),)),
            n["a2"]: TensorSpec((qd, spec.rank), free=((1, "a1"),)),
            n["a2_bias"]: TensorSpec((qd,), init="uniform:-1:2", role="vector"),
        }

    @classmethod
    def cache_need(cls, spec):
        return StateNeed((spec.heads, spec.dim, spec.vdim), "float32")

    def __init__(self, spec, weights: Dict[str, torch.Tensor], rt):
        if not spec.tau > 0:
            raise ValueError(f"gla: tau {spec.tau} must be positive")
        n, f32 = spec.names, torch.float32
        self._setup(spec, rt, spec.vdim, weights[n["norm"]].to(f32).reshape(1, spec.vdim).repeat(spec.heads, 1).reshape(-1), weights[n["o"]])
        self.w_in = rt.matrix(torch.cat([weights[n[k]].to(f32) for k in ("q", "k", "v", "gate")], 0))
        a1 = weights[n["a1"]].to(f32)
        self.rank = a1.shape[0]
        pad = (-self.rank) % 16                    # (whole 16-row tiles of the few-row product)
        if pad:
            a1 = torch.cat([a1, torch.zeros(pad, a1.shape[1])], 0)
        self.w_a1, self.w_a2 = rt.matrix(a1), rt.matrix(weights[n["a2"]])
        self.b_a2 = rt.vector(weights[n["a2_bias"]])

    def takes_prenormed(self, rows: int) -> bool:
        return self.rt.few_rows_shape(rows, self.w_in) and self.rt.few_rows_shape(rows, self.w_a1) and self.w_in.shape[1] % 8 == 0

    def heads(self, x, step, cache, out) -> None:
        s, rt = self.spec, self.rt
        if cache is None or len(cache) != 1 or not cache.owner:
            raise RuntimeError("gated linear attention keeps its own memory")
        T, qd, vd = x.shape[0], s.heads * s.dim, s.heads * s.vdim
        proj = rt.linear(x, self.w_in, "gla_proj")
        hidden = rt.linear(x, self.w_a1, "gla_hidden", out_dtype=torch.float32)
        decay = rt.ws.get("memory_decay", (T, qd), torch.float32)
        ops.low_rank_decay(hidden, self.w_a2, self.b_a2, decay, "rooted_sigmoid", power=1.0 / s.tau)
        self._scan(proj, proj[:, qd:], proj[:, 2 * qd:], decay, cache.storage, proj[:, 2 * qd + vd:], out, step, float(s.dim) ** -0.5)


class TimeMixingMixer(DecayMemoryMixer):
    kind = "time_mixing"

    @classmethod
    def tensors(cls, spec) -> Dict[str, TensorSpec]:
        n, D, W = spec.names, spec.heads * spec.dim, spec.hidden
        out = {n[f"mu_{s}"]: TensorSpec((W,), init="uniform:0:1", role="vector") for s in "rkvgw"}
        for key in ("r", "k", "v", "gate"):
            out[n[key]] = TensorSpec((D, W))
        out.update({
            n["w1"]: TensorSpec((spec.rank, W), free=((0, "w1"),)), n["w2"]: TensorSpec((D, spec.rank), free=((1, "w1"),)),
            n["w0"]: TensorSpec((D,), init="uniform:-6:0", role="vector"),
            n["u"]: TensorSpec((spec.heads, spec.dim), init="uniform:-1:1", role="vector"),
            n["norm"]: TensorSpec((D,), init="ones", role="vector"), n["o"]: TensorSpec((W, D)),
        })
        return out

    @classmethod
    def cache_need(cls, spec):
        return StateNeed((spec.hidden,), "compute"), StateNeed((spec.heads, spec.dim, spec.dim), "float32")

    def __init__(self, spec, weights: Dict[str, torch.Tensor], rt):
        n, f32 = spec.names, torch.float32
        self._setup(spec, rt, spec.dim, weights[n["norm"]].to(f32), weights[n["o"]])
        self.mu = rt.vector(torch.stack([weights[n[f"mu_{s}"]].to(f32).reshape(-1) for s in "rkvgw"]))
        self.w_in = rt.matrix(torch.stack([weights[n[k]].to(f32) for k in ("r", "k", "v", "gate")]))     # [4, heads * dim, hidden]
        w1 = weights[n["w1"]].to(f32)
        pad = (-w1.shape[0]) % 16
        if pad:
            w1 = torch.cat([w1, torch.zeros(pad, w1.shape[1])], 0)
        self.w_1, self.w_2 = rt.matrix(w1), rt.matrix(weights[n["w2"]])
        self.w_0 = rt.vector(weights[n["w0"]].to(f32).reshape(-1))
        self.bonus = rt.vector(weights[n["u"]].to(f32).reshape(-1))

    def heads(self, x, step, cache, out) -> None:
        s, rt = self.spec, self.rt
        if cache is None or len(cache) != 2 or not cache.owner:
            raise RuntimeError("time mixing keeps its own last input and memory")
        T, W, D = x.shape[0], s.hidden, s.heads * s.dim
        mixes = rt.ws.get("token_mixes", (5, T, W), rt.act_dtype)
        ops.token_mix(x, cache[0].storage, self.mu, mixes, step.seq_of_token, step.cu_seqlens, step.slots)
        rkvg = rt.ws.get("time_rkvg", (4, T, D), rt.act_dtype)
        if rt.few_rows(mixes[0], self.w_in[0]):
            for i in range(4):
                rt.few_rows_product(mixes[i], self.w_in[i], rkvg[i])
        else:
            rt.batched_product(mixes[:4], self.w_in, rkvg)
        hidden = rt.linear(mixes[4], self.w_1, "time_hidden", out_dtype=torch.float32)
        decay = rt.ws.get("memory_decay", (T, D), torch.float32)
        ops.low_rank_decay(hidden, self.w_2, self.w_0, decay, "double_exp", hidden_tanh=True)
        self._scan(rkvg[0], rkvg[1], rkvg[2], decay, cache[1].storage, rkvg[3], out, step, 1.0, bonus=self.bonus)


registry.register_mixer(GatedLinearMixer.kind, GatedLinearMixer)
registry.register_mixer(TimeMixingMixer.kind, TimeMixingMixer)
