"""A token's own input to a layer, behind the layer's feed-forward:

    e = D[tok][layer * dim : (layer + 1) * dim]       D the model's side table [vocab, layers * dim]
    x <- x + rms(W_proj (act(W_gate x) * e)) * w      rms over the width, float32

W_gate reads the stream itself (no norm in front of it).  A step of a few rows makes the gated middle in one launch, straight
from the float32 stream; more rows take the stream in the activations' dtype, the product, and one launch that applies the
activation and the token's part.  The norm, the sum and the norm that reads the stream next are one kernel (``branch_norm``).
The table belongs to the model, which hands it over with ``attach``; dim, eps and the activation are the spec's.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..config.specs import NormSpec
from ..weights.loader import TensorSpec
from .linear import Linear
from .norm import RMSNorm, RowsInfo


class TokenSide:
    def __init__(self, spec, layer: int, hidden: int, rt):
        from ..kernels import ACTIVATIONS
        if spec.dim <= 0 or spec.activation not in ACTIVATIONS or ACTIVATIONS[spec.activation] > 3:
            raise ValueError(f"token_side: {spec.dim} values a layer with activation '{spec.activation}'")
        self.spec, self.layer, self.hidden, self.rt = spec, layer, hidden, rt
        self.dim, self.act = int(spec.dim), ACTIVATIONS[spec.activation]
        self.norm = RMSNorm(NormSpec(kind="rmsnorm", size=hidden, eps=spec.eps), rt)
        self.gate = self.proj = self.table = None

    @staticmethod
    def _n(prefix, names, key):
        return f"{prefix}{names[key]}{names.get('suffix', '.weight')}"

    def plan(self, prefix: str, names: Dict[str, str]) -> Dict[str, TensorSpec]:
        p = {self._n(prefix, names, "side_gate"): TensorSpec((self.dim, self.hidden)),
             self._n(prefix, names, "side_proj"): TensorSpec((self.hidden, self.dim), std=self.dim ** -0.5)}
        p.update(self.norm.plan(self._n(prefix, names, "side_norm")))
        return p

    def load(self, tensors, prefix: str, names: Dict[str, str]) -> None:
        self.gate = Linear(tensors[self._n(prefix, names, "side_gate")], None, self.rt)
        self.proj = Linear(tensors[self._n(prefix, names, "side_proj")], None, self.rt)
        self.norm.load(tensors, self._n(prefix, names, "side_norm"))

    def attach(self, table: torch.Tensor) -> None:
        if table.shape[1] < (self.layer + 1) * self.dim:
            raise ValueError(f"token_side: a side table of {table.shape[1]} values a token holds no part of {self.dim} for layer {self.layer}")
        self.table = table

    def state(self, prefix: str, names: Dict[str, str]) -> Dict[str, torch.Tensor]:
        out = {self._n(prefix, names, "side_gate"): self.gate.weight, self._n(prefix, names, "side_proj"): self.proj.weight}
        out.update(self.norm.state(self._n(prefix, names, "side_norm")))
        return out

    def nbytes(self) -> int:
        return self.gate.nbytes() + self.proj.nbytes() + self.norm.nbytes()

    def scratch_row(self) -> int:
        return 2 * self.dim + 3 * self.hidden

    graph_safe = True

    def forward(self, x: torch.Tensor, batch, next_norm=None):
        """Adds into x; with ``next_norm`` (an ``RMSNorm`` of the model's width) its rows come back in a ``RowsInfo``."""
        K_, rt = self.rt.kernels, self.rt
        rows, col = x.shape[0], self.layer * self.dim
        z = rt.empty(rows, self.dim)
        if rows <= getattr(K_, "SIDE_FEW_ROWS", 0):
            K_.token_side_few(x, self.gate.weight, self.table, batch.tokens, col, z, self.act)
        else:
            if rt.full_precision:
                h = x
            else:
                h = rt.empty(*x.shape)
                K_.cast_rows(x, h)
            self.gate.store(h, z)
            K_.token_side_apply(z, self.table, batch.tokens, col, self.act)
        y = self.proj.logits(z)
        if next_norm is not None and (getattr(next_norm, "weight", None) is None or next_norm.spec.kind != "rmsnorm"
                                      or next_norm.spec.size != self.hidden):
            next_norm = None
        h = rt.empty(*x.shape) if next_norm is not None else None
        K_.branch_norm(x, y, self.norm.weight, self.norm.spec.eps, h, (next_norm.weight, next_norm.spec.eps) if next_norm is not None else None)
        return RowsInfo(norm=next_norm, h=h) if next_norm is not None else None
