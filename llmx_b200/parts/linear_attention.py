"""Decayed linear attention: a matrix state per head instead of a cache of keys.

For the rows of a step, per head h with key width D and value width V:
    q, k = silu(h Wq^T), silu(h Wk^T)      [heads, D]
    v    = silu(h Wv^T)                    [heads, V]
    S_t  = decay_h S_{t-1} + k_t v_t^T     (32-bit, one [D, V] matrix per request and head, in a state slot)
    o_t  = S_t^T q_t                       (no other scale)
    y    = RMSNorm over all heads' outputs together (weight of heads * V) * sigmoid(h Wg^T)
    residual += y Wo^T
The per-head decays are constants of the architecture's configuration.  The four input projections are one product
over the stacked weight; the activation, the recurrence (csrc/recurrence.cu) and the gated norm (csrc/rowwise.cu)
are kernels of their own; the recurrence has a form for steps of a row or a few and one for long portions.

Options for designs that vary it (retention is `activation=None, rot_dims, key_factor, norm="heads", gate="silu"`):
    activation None    q, k and v enter the recurrence as projected
    rot_dims           the first `rot_dims` values of every q and k head are turned by the row's position, pair
                       (i, i + rot_dims / 2) by p * rot_base^(-2i / rot_dims) (after the activation)
    key_factor         a factor on k (after the rotation)
    norm "heads"       every head's output divided by its own root mean square, no weight (no tensor `norm`)
    gate "silu"        silu instead of sigmoid
"""
from __future__ import annotations

from typing import Dict, Optional, Sequence

import numpy as np
import torch

from .. import ops, runtime
from ..cache.manager import StateSpec
from ..weights.spec import TensorSpec
from .base import Part, Precision, StepBatch
from .linear import Linear, stored_product
from .rope import power_frequencies


class DecayedLinearAttention(Part):
    def __init__(self, hidden: int, heads: int, key_dim: int, value_dim: int, decay: Sequence[float], norm_eps: float,
                 names=("q", "k", "v", "g", "o", "norm"), activation: Optional[str] = "silu", rot_dims: int = 0, rot_base: float = 10000.0,
                 key_factor: float = 1.0, norm: str = "row", gate: str = "sigmoid"):
        if len(decay) != heads:
            raise ValueError("decayed linear attention: one decay per head")
        if activation not in (None, "silu") or norm not in ("row", "heads") or gate not in ("sigmoid", "silu"):
            raise ValueError("decayed linear attention: activation silu or None, norm over the row or per head, gate sigmoid or silu")
        if rot_dims % 2 or not 0 <= rot_dims <= key_dim:
            raise ValueError("decayed linear attention: the rotated width must be even and at most the key width")
        self.activation, self.norm_kind, self.gate = activation, norm, gate
        self.rot_dims, self.rot_base, self.key_factor = int(rot_dims), float(rot_base), float(key_factor)
        self.freq: Optional[torch.Tensor] = None
        self.hidden, self.heads, self.key_dim, self.value_dim = int(hidden), int(heads), int(key_dim), int(value_dim)
        self.decay_values = [float(d) for d in decay]
        self.norm_eps, self.names = float(norm_eps), tuple(names)
        self.qk_width, self.v_width = self.heads * self.key_dim, self.heads * self.value_dim

    def stored_products(self):
        """The products whose result is stored (not added to the residual): a block may clear their outputs in passing."""
        return (self.inputs,)

    def cache_spec(self):
        return StateSpec((self.heads * self.value_dim * self.key_dim,), "float32")

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        q, k, v, g, o, norm = self.names
        specs = {q: TensorSpec((self.qk_width, self.hidden)), k: TensorSpec((self.qk_width, self.hidden)),
                 v: TensorSpec((self.v_width, self.hidden)), g: TensorSpec((self.v_width, self.hidden)),
                 o: TensorSpec((self.hidden, self.v_width))}
        if self.norm_kind == "row":
            specs[norm] = TensorSpec((self.v_width,), "vector", init="one_plus_normal", std=0.01)
        return specs

    def load(self, tensors, precision: Precision) -> None:
        super().load(tensors, precision)
        self.cleared_outputs = {}
        q, k, v, g, o, norm = self.names
        self.inputs = Linear(torch.cat([tensors[q], tensors[k], tensors[v], tensors[g]], dim=0), precision)
        self.o = Linear(tensors[o], precision)
        self.norm_weight = tensors[norm].to(torch.float32).contiguous() if self.norm_kind == "row" else None
        device = tensors[o].device
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=device)
        # Frequencies in double precision, rounded once; the angle is the float product with the position.
        self.freq = torch.from_numpy(power_frequencies(self.rot_base, self.rot_dims).astype(np.float32)).to(device) if self.rot_dims else None

    def forward(self, h: torch.Tensor, step: StepBatch, cache_entry: int, residual: torch.Tensor,
                write_cache: bool = True) -> None:
        rows = h.shape[0]
        if not (h.is_cuda and h.is_contiguous() and h.dtype is self.precision.act and tuple(h.shape) == (rows, self.hidden)
                and residual.dtype is torch.float32 and residual.is_contiguous() and tuple(residual.shape) == (rows, self.hidden)):
            raise runtime.KernelError("linear attention: rows of the path's type and the mixer's width, a float32 residual")
        qk, vw = self.qk_width, self.v_width
        proj = stored_product(self, self.inputs, h)                                             # [rows, q | k | v | g]
        if self.activation == "silu":
            ops.silu_columns_(proj, 0, 2 * qk + vw)
        if self.rot_dims or self.key_factor != 1.0:
            ops.rotate_heads_(proj, self.heads, self.heads, self.key_dim, self.rot_dims, self.freq, step.positions, 1.0, self.key_factor)
        o = torch.empty((rows, vw), dtype=torch.float32, device=h.device)
        ops.linear_recurrence(proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:2 * qk + vw], step.state(cache_entry), step, o,
                              self.heads, self.heads, self.key_dim, self.value_dim, decay=self.decay)
        y = torch.empty((rows, vw), dtype=self.precision.act, device=h.device)
        group = vw if self.norm_kind == "row" else self.value_dim
        ops.gated_rmsnorm(o, proj[:, 2 * qk + vw:], self.norm_weight, self.norm_eps, group, self.gate, y)
        self.o(y, out=residual, accumulate=True)
