"""Mixers that keep a float32 matrix a head as their memory and read it with a query.

``gated_linear_attention`` (a decay a key channel):
    q = W_q h * dim^(-1/2), k = W_k h  [heads, dim];   v = W_v h  [heads, v_dim]
    a = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)           one a head and key channel, through a low rank
    S_t = diag(a_t) S_(t-1) + k_t v_t^T;               o_t = S_t^T q_t
    y   = W_o ( rms(o over a head's values) * w * silu(W_g h) )          w [v_dim], one for all heads

``mlstm`` (one input gate and one forget gate a head, exponential, with a running maximum m):
    q, k, v as above;   i = cap tanh((W_i h + b_i) / cap);   f = log sigmoid(cap tanh((W_f h + b_f) / cap))
    m_t = max(f_t + m_(t-1), i_t);   S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T;   n_t likewise with k_t
    o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)
    y   = W_o ( rms(o over a head's values) * w * sigmoid(W_g h) )       w [heads * v_dim]

All states (S; for ``mlstm`` also n and m) are float32, start at zero and travel with the sequence (``StateRequest``s); a step
walks its rows in order from the state the steps before left, so prompts, pieces of prompts and single tokens are one
path.  Every projection of h is a row block of one matrix; a step of few rows keeps the whole product's result in float32,
a longer one stores it in the activations' dtype (the input and forget gates in float32 even then, as a product of their
own rows).  Decays, gates, the recurrence and the norm behind it are float32.  Sizes, ``tau``, ``gate_cap``, the rank and
the norm's ``eps`` are the spec's.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..cache.kv import StateRequest
from ..weights.loader import TensorSpec
from .linear import Linear, SKINNY_ROWS
from .registry import register_mixer

NORMALIZER_EPS = 1e-6       # of the mlstm read-out's denominator


class MatrixMemory:
    """What the two mixers share: sizes, the stacked projection, the norm with its gate, the output product."""

    KIND = ""
    EXTRA = ()                   # keys of the row blocks behind q | k | v | g

    def __init__(self, spec, layer: int, rt):
        p = spec.params
        self.heads, self.dim, self.vdim = spec.n_heads, spec.head_dim, int(p["v_dim"])
        self.eps = float(p["eps"])
        if min(self.heads, self.dim, self.vdim) <= 0 or self.dim > 256:
            raise ValueError(f"{self.KIND}: heads {self.heads}, key size {self.dim} (at most 256) and value size {self.vdim} must be positive")
        self.spec, self.layer, self.rt = spec, layer, rt
        self.qd, self.vd = self.heads * self.dim, self.heads * self.vdim
        self.main = 2 * self.qd + 2 * self.vd                          # columns of q | k | v | g
        self.proj = self.out = self.norm = None
        self.vectors: Dict[str, torch.Tensor] = {}

    # ------------------------------------------------------------------ weights
    @staticmethod
    def _n(prefix, names, key):
        return f"{prefix}{names[key]}{names.get('suffix', '.weight')}"

    def _rows(self) -> Dict[str, int]:
        """Rows of every block of the stacked projection, in its order."""
        raise NotImplementedError

    def _vectors(self) -> Dict[str, TensorSpec]:
        raise NotImplementedError

    def plan(self, prefix: str, names: Dict[str, str]) -> Dict[str, TensorSpec]:
        H = self.spec.hidden
        p = {self._n(prefix, names, k): TensorSpec((rows, H)) for k, rows in self._rows().items()}
        p[self._n(prefix, names, "o")] = TensorSpec((H, self.vd))
        for k, s in self._vectors().items():
            p[self._n(prefix, names, k)] = s
        return p

    def load(self, tensors, prefix: str, names: Dict[str, str]) -> None:
        pieces = [tensors[self._n(prefix, names, k)] for k in self._rows()]
        pad = -sum(t.shape[0] for t in pieces) % 8                     # a row of the result keeps its 16-byte alignment
        if pad:
            pieces.append(torch.zeros((pad, self.spec.hidden), dtype=pieces[0].dtype, device=pieces[0].device))
        self.proj = Linear(pieces, None, self.rt)
        self.out = Linear(tensors[self._n(prefix, names, "o")], None, self.rt)
        self.vectors = {k: self.rt.vector(tensors[self._n(prefix, names, k)]) for k in self._vectors()}
        self.norm = self.vectors["norm"]

    def state(self, prefix: str, names: Dict[str, str]) -> Dict[str, torch.Tensor]:
        out, r = {}, 0
        for k, rows in self._rows().items():
            out[self._n(prefix, names, k)] = self.proj.weight[r:r + rows]
            r += rows
        out[self._n(prefix, names, "o")] = self.out.weight
        for k, t in self.vectors.items():
            out[self._n(prefix, names, k)] = t
        return out

    def nbytes(self) -> int:
        return self.proj.nbytes() + self.out.nbytes() + 4 * sum(t.numel() for t in self.vectors.values())

    def scratch_row(self) -> int:
        # the projection's row, the recurrence's float32 output and decays, the gated row, and a long step's share of the
        # segments' states (a state a segment of some hundred tokens)
        return self.main + 3 * self.vd + 2 * self.qd + self.heads * self.dim * self.vdim // 64

    graph_safe = True

    # ------------------------------------------------------------------ cache
    @classmethod
    def state_name(cls, site: int, what: str = "") -> str:
        return f"{cls.KIND}.{site}{'.' + what if what else ''}"

    def cache_requests(self, site: int) -> List[object]:
        return [StateRequest(self.state_name(site), (self.heads, self.dim, self.vdim), torch.float32)]

    # ------------------------------------------------------------------ step
    def forward(self, h, x: torch.Tensor, batch, cache, site: int, next_norm=None):
        return self.out.accumulate(self._gated(h, batch, cache, site), x, next_norm)

    def produce(self, h, batch, cache, site: int) -> torch.Tensor:
        """The mixer's output as float32 rows of its own (what ``forward`` adds into x)."""
        return self.out.logits(self._gated(h, batch, cache, site))

    def _project(self, h) -> torch.Tensor:
        """[rows, q | k | v | g | ...]: float32 for few rows, else in the activations' dtype."""
        if h.shape[0] <= SKINNY_ROWS:
            return self.proj.logits(h)
        return self.proj.store(h)

    def _split(self, p):
        qd, vd = self.qd, self.vd
        return p[:, :qd], p[:, qd:2 * qd], p[:, 2 * qd:2 * qd + vd], p[:, 2 * qd + vd:self.main]

    def _gated(self, h, batch, cache, site: int) -> torch.Tensor:
        raise NotImplementedError


class GatedLinearAttention(MatrixMemory):
    KIND = "gated_linear_attention"

    def __init__(self, spec, layer: int, rt):
        super().__init__(spec, layer, rt)
        self.tau, self.rank = float(spec.params["tau"]), int(spec.params["rank"])
        if self.tau <= 0 or not (0 < self.rank <= 1024):
            raise ValueError(f"{self.KIND}: tau {self.tau} must be positive and the rank {self.rank} lie in 1..1024")
        self.a2 = None

    def _rows(self):
        return {"q": self.qd, "k": self.qd, "v": self.vd, "g": self.vd, "a1": self.rank}

    def _vectors(self):
        return {"norm": TensorSpec((self.vdim,), init="ones_normal"), "a2_bias": TensorSpec((self.qd,), std=1.0)}

    def plan(self, prefix, names):
        p = super().plan(prefix, names)
        p[self._n(prefix, names, "a2")] = TensorSpec((self.qd, self.rank), std=0.1)
        return p

    def load(self, tensors, prefix, names):
        super().load(tensors, prefix, names)
        self.a2 = self.rt.matrix(tensors[self._n(prefix, names, "a2")])

    def state(self, prefix, names):
        out = super().state(prefix, names)
        out[self._n(prefix, names, "a2")] = self.a2
        return out

    def nbytes(self) -> int:
        return super().nbytes() + self.a2.numel() * self.a2.element_size()

    def _gated(self, h, batch, cache, site: int) -> torch.Tensor:
        K_, rt = self.rt.kernels, self.rt
        if hasattr(h, "tensor"):
            h = h.tensor()
        rows = h.shape[0]
        p = self._project(h)
        q, k, v, gate = self._split(p)
        decay = rt.empty(rows, self.qd, dtype=torch.float32)
        K_.channel_decay(p[:, self.main:self.main + self.rank], self.a2, self.vectors["a2_bias"], self.tau, decay)
        o = rt.empty(rows, self.vd, dtype=torch.float32)
        K_.memory(q, k, v, decay, cache.state[self.state_name(site)], batch, o, self.heads, self.dim, self.vdim, self.dim ** -0.5)
        out = rt.empty(rows, self.vd)
        K_.group_rmsnorm_gate(o, self.norm, gate, out, self.heads, self.eps, silu=True)
        return out


class MLSTM(MatrixMemory):
    KIND = "mlstm"

    def __init__(self, spec, layer: int, rt):
        super().__init__(spec, layer, rt)
        self.cap = float(spec.params["gate_cap"])
        if self.cap <= 0:
            raise ValueError(f"{self.KIND}: gate_cap {self.cap} must be positive")
        self.gates = None                                              # the gates' rows of the projection as a product of their own

    def _rows(self):
        return {"q": self.qd, "k": self.qd, "v": self.vd, "g": self.vd, "i": self.heads, "f": self.heads}

    def _vectors(self):
        return {"norm": TensorSpec((self.vd,), init="ones_normal"), "i_bias": TensorSpec((self.heads,), std=1.0),
                "f_bias": TensorSpec((self.heads,), std=1.0)}

    def load(self, tensors, prefix, names):
        super().load(tensors, prefix, names)
        self.gates = Linear(self.proj.weight[self.main:], None, self.rt)            # (a view: contiguous rows of the one matrix)

    def cache_requests(self, site: int) -> List[object]:
        return super().cache_requests(site) + [StateRequest(self.state_name(site, "n"), (self.heads, self.dim), torch.float32),
                                               StateRequest(self.state_name(site, "m"), (self.heads,), torch.float32)]

    def _gated(self, h, batch, cache, site: int) -> torch.Tensor:
        K_, rt = self.rt.kernels, self.rt
        if hasattr(h, "tensor"):
            h = h.tensor()
        rows, f32 = h.shape[0], torch.float32
        p = self._project(h)
        q, k, v, gate = self._split(p)
        z = p[:, self.main:] if p.dtype is f32 else self.gates.logits(h)
        ab, low = rt.empty(rows, self.heads, 2, dtype=f32), rt.empty(rows, self.heads, dtype=f32)
        K_.scalar_gates(z, self.vectors["i_bias"], self.vectors["f_bias"], self.cap, cache.state[self.state_name(site, "m")], batch, ab, low)
        o, den = rt.empty(rows, self.vd, dtype=f32), rt.empty(rows, self.heads, dtype=f32)
        K_.memory(q, k, v, ab, cache.state[self.state_name(site)], batch, o, self.heads, self.dim, self.vdim, self.dim ** -0.5,
                  norm_state=cache.state[self.state_name(site, "n")], norm_out=den)
        out = rt.empty(rows, self.vd)
        K_.group_rmsnorm_gate(o, self.norm, gate, out, self.heads, self.eps, divisor=(den, low, NORMALIZER_EPS))
        return out


register_mixer(GatedLinearAttention.KIND, GatedLinearAttention)
register_mixer(MLSTM.KIND, MLSTM)
