"""Gated linear attention: a matrix state per head whose rows (key channels) are decayed each by a gate the token chooses.

For the rows of a step, with H heads of key width D and value width V:
    q = h Wq^T * D^-1/2,  k = h Wk^T      [heads, D]        v = h Wv^T      [heads, V]
    alpha = sigmoid(Wa2 (Wa1 h) + b)^(1 / tau)              [heads, D], through a low-rank pair
    S_t = diag(alpha_t) S_{t-1} + k_t v_t^T                 (32-bit, one [D, V] matrix per request and head, in a state slot)
    o_t = S_t^T q_t                                         (the read sees the write)
    y   = RMSNorm per head over V (one weight of V shared by the heads) * silu(h Wg^T)
    residual += y Wo^T
Whatever reads h is one product over the stacked weight (the low-rank pair's inner values are its last columns); the pair's
second product, its bias, the decay and q's factor are one 32-bit kernel and the recurrence another (csrc/recurrence.cu), the
gated norm a third (csrc/rowwise.cu).  Tensor roles: q, k, v, g, o, norm, a1 [rank, E], a2 [heads * D, rank], a2.b.  A rank of
-1 stands for "whatever the stored tensors have".
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops, runtime
from ..cache.manager import StateSpec
from ..weights.spec import TensorSpec
from .base import Part, Precision, StepBatch
from .linear import Linear, add_product, stored_product


class GatedLinearAttention(Part):
    def __init__(self, hidden: int, heads: int, key_dim: int, value_dim: int, tau: float, norm_eps: float, decay_rank: int = -1):
        if not tau > 0:
            raise ValueError("gated linear attention: the root taken of the decay must be positive")
        if decay_rank == 0 or decay_rank < -1:
            raise ValueError("gated linear attention: the decay's rank is positive, or -1 for the stored tensors'")
        self.hidden, self.heads, self.key_dim, self.value_dim = int(hidden), int(heads), int(key_dim), int(value_dim)
        self.tau, self.norm_eps, self.decay_rank = float(tau), float(norm_eps), int(decay_rank)
        self.qk_width, self.v_width = self.heads * self.key_dim, self.heads * self.value_dim

    def stored_products(self):
        """The products whose result is stored (not added to the residual): a block may clear their outputs in passing."""
        return (self.inputs,)

    def output_product(self) -> Linear:
        return self.o

    def cache_spec(self):
        return StateSpec((self.heads * self.value_dim * self.key_dim,), "float32")

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        E = self.hidden
        return {"q": TensorSpec((self.qk_width, E)), "k": TensorSpec((self.qk_width, E)), "v": TensorSpec((self.v_width, E)),
                "g": TensorSpec((self.v_width, E)), "o": TensorSpec((E, self.v_width)),
                "norm": TensorSpec((self.value_dim,), "vector", init="one_plus_normal", std=0.01),
                "a1": TensorSpec((self.decay_rank, E)), "a2": TensorSpec((self.qk_width, self.decay_rank), std=0.1),
                "a2.b": TensorSpec((self.qk_width,), "vector", std=0.5)}

    def load(self, tensors, precision: Precision) -> None:
        super().load(tensors, precision)
        self.cleared_outputs = {}
        t = tensors
        self.decay_rank = int(t["a1"].shape[0])
        if t["a2"].shape[1] != self.decay_rank:
            raise ValueError("gated linear attention: the decay's two low-rank matrices do not fit each other")
        self.inputs = Linear(torch.cat([t["q"], t["k"], t["v"], t["g"], t["a1"]], dim=0), precision)
        self.o = Linear(t["o"], precision)
        self.a2t = t["a2"].to(torch.float32).t().contiguous()             # [rank, heads * D]: neighbouring channels are one read
        self.a2_bias = t["a2.b"].to(torch.float32).contiguous()
        self.norm_weight = t["norm"].to(torch.float32).contiguous()

    def forward(self, h: torch.Tensor, step: StepBatch, cache_entry: int, residual: torch.Tensor,
                write_cache: bool = True) -> None:
        rows = h.shape[0]
        if not (h.is_cuda and h.is_contiguous() and h.dtype is self.precision.act and tuple(h.shape) == (rows, self.hidden)
                and residual.dtype is torch.float32 and residual.is_contiguous() and tuple(residual.shape) == (rows, self.hidden)):
            raise runtime.KernelError("gated linear attention: rows of the path's type and the mixer's width, a float32 residual")
        qk, vw = self.qk_width, self.v_width
        g_off = 2 * qk + vw
        proj = stored_product(self, self.inputs, h)                            # [rows, q | k | v | g | a1]
        decay = torch.empty((rows, qk), dtype=torch.float32, device=h.device)
        ops.channel_decay_(proj, g_off + vw, self.a2t, self.a2_bias, self.tau, decay, 0, self.key_dim ** -0.5)
        o = torch.empty((rows, vw), dtype=torch.float32, device=h.device)
        ops.linear_recurrence(proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:g_off], step.state(cache_entry), step, o, self.heads,
                              self.heads, self.key_dim, self.value_dim, gate=decay, form="channel")
        y = torch.empty((rows, vw), dtype=self.precision.act, device=h.device)
        ops.gated_rmsnorm(o, proj[:, g_off:g_off + vw], self.norm_weight, self.norm_eps, self.value_dim, "silu", y)
        add_product(self, self.o, y, residual)
