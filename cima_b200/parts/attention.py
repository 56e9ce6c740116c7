"""Grouped-query causal attention over the paged cache, with optional window.

forward: qkv = h Wqkv^T + b  ->  rotate q, k and append k, v to the layer's pages  ->
attention (prefill: over the step's own keys; decode: over the cache)  ->  x += att Wo^T.
Formulas and order as the reference's layer loop, steps 2-7 (src/models/transformer.rs:1039-1264):
bias before rotation, rotation before caching, scale = spec.scale, head h reads kv head
h / (heads / kv_heads), no output bias unless the spec says so.

Every size (heads, kv heads, head_dim, window, scale, bias flags) is a field of the spec.  More are ``params``:
``v_dim``, a value size that differs from the key size, and ``sink``, a number of entries of score 0 that carry no
value and join every row's softmax denominator (1: p_j = exp(s_j) / (1 + sum exp(s))); ``keep_first``: with a window, a
sequence's first so many positions stay visible below it, at their own positions (such a layer keeps every page: a ring
would hand the first pages on).  A position encoding whose pairs are neighbours (``interleaved``) is served by
permuting the rows of W_q and W_k at load, alike in every head, which leaves every score as it is; a position
encoding's ``amplitude`` multiplies sine and cosine in the rotating kernel.  ``qk_norm_eps`` e: every head of q and k is divided
by its root mean square over its ``head_dim`` values (e inside the root, no weight) before the rotation and the cache;
``q_temp`` (coef, every): the queries at position p are then multiplied by 1 + coef ln(floor((p + 1) / every) + 1);
``head_sink``: a stored number a head (tensor "sink") whose exponential joins that head's denominator, neither scaled nor
attached to a value; ``gate``: the heads' results leave times sigmoid(W_g h), value by value (tensor "g", whose rows stand
behind q | k | v in the same product, so that a row's gate lies in its own buffer and the attention kernels apply it where
they finish a row).  ``row_norm_eps`` e: the whole q projection of a row (all its heads at once) is divided by its root mean
square and multiplied by a weight of its size (tensor "q_norm"), and so is the whole k projection ("k_norm"), before the cache;
``distance_slopes``, one number a head: m_h (i - j) is taken off the scaled score of position i with position j; ``v_mix``: the
layer named "first" leaves its values to the later layers of the step, one named "mix" uses (1 - l) v + l v_first with the
stored number l (tensor "v_mix") and caches that.  ``own_kv`` False goes with ``cache_from``: the layer stores no W_k and W_v.  Keys and values live in the
cache at one size, the larger of the two rounded up to 16: the rows of W_q, W_k, W_v (and the columns of W_o) that
pad a head are zero, so scores and outputs are what the unpadded sizes give.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..cache.kv import KVRequest
from ..weights.loader import TensorSpec
from .linear import Linear
from .registry import build_position, register_mixer


FIRST_VALUES = "attention.first_values"      # of ``StepBatch.carried``: (rows of values, values of a head there)


class Attention:
    def __init__(self, spec, layer: int, rt):
        self.dim, self.vdim = spec.head_dim, int(spec.params.get("v_dim", spec.head_dim))
        self.sink = float(spec.params.get("sink", 0.0))
        self.keep_first = int(spec.params.get("keep_first", 0)) if spec.window else 0
        self.qk_eps = spec.params.get("qk_norm_eps")
        self.q_temp = spec.params.get("q_temp")
        self.has_sink, self.gated = bool(spec.params.get("head_sink", False)), bool(spec.params.get("gate", False))
        self.own_kv = bool(spec.params.get("own_kv", True))
        self.row_eps, self.v_mix = spec.params.get("row_norm_eps"), spec.params.get("v_mix")
        self.slopes_host = spec.params.get("distance_slopes")
        if not self.own_kv and spec.cache_from is None:
            raise ValueError("attention: a layer without keys and values of its own names the site whose cache it reads")
        if self.sink and self.has_sink:
            raise ValueError("attention: a sink is either a number of entries of score 0 or a stored number a head")
        self.padded = self.dim != self.vdim or self.dim % 16 != 0
        self.hd = -(-max(self.dim, self.vdim) // 16) * 16 if self.padded else self.dim      # a head's size in a step's rows and in the cache
        if min(self.dim, self.vdim) <= 0 or self.hd > 256:
            raise ValueError(f"attention: key size {self.dim} and value size {self.vdim} must be positive, at most 256")
        if spec.n_heads % spec.n_kv_heads:
            raise ValueError(f"attention: {spec.n_heads} heads are not a multiple of {spec.n_kv_heads} kv heads")
        if (self.gated or not self.own_kv) and (spec.qkv_bias or spec.out_bias):
            raise ValueError("attention: biases beside an output gate or another layer's keys and values are not implemented")
        if self.padded and (spec.qkv_bias or spec.out_bias) and spec.position.rotary_dim:
            raise ValueError(f"attention: head_dim {self.dim} must be a multiple of 16 and equal to the value size {self.vdim} "
                             f"where biased projections rotate (their heads are padded in the cache only without rotation)")
        if self.v_mix not in (None, "first", "mix"):
            raise ValueError(f"attention: v_mix '{self.v_mix}' is neither 'first' nor 'mix'")
        if self.slopes_host is not None and len(self.slopes_host) != spec.n_heads:
            raise ValueError(f"attention: {len(self.slopes_host)} distance slopes for {spec.n_heads} heads")
        if self.row_eps is not None or self.v_mix is not None:
            if spec.cache_from is not None or self.qk_eps or self.q_temp or self.gated or (spec.position is not None and spec.position.rotary_dim):
                raise ValueError("attention: a norm over the whole projection and mixed values go with keys and values of the layer's own and "
                                 "without rotation, head norms, query temperature or gate")
            if self.row_eps is None:
                raise ValueError("attention: mixed values go with the norm over the whole projection (one kernel does both)")
        self.spec, self.layer, self.rt = spec, layer, rt
        self.position = build_position(spec.position, rt)
        # (a position part registered elsewhere may offer neither: half-split pairs, amplitude 1)
        self.interleaved = bool(getattr(self.position, "interleaved", False))
        self.amplitude = float(getattr(self.position, "amplitude", 1.0))
        self.qd = spec.n_heads * self.hd
        self.nk = spec.n_kv_heads if self.own_kv else 0                  # key (and value) heads of a step's rows
        self.kvd = self.nk * self.hd
        self.gate_col = self.qd + 2 * self.kvd if self.gated else 0      # where a row's gate begins
        self.qkv = None
        self.out = None
        self.sinks = self.slopes = self.q_weight = self.k_weight = self.mix = None

    # ------------------------------------------------------------------ weights
    def plan(self, prefix: str, names: Dict[str, str]) -> Dict[str, TensorSpec]:
        s = self.spec
        sfx = names.get("suffix", ".weight")
        p: Dict[str, TensorSpec] = {}
        for key, heads, size in self._pieces():
            rows = heads * size
            p[f"{prefix}{names[key]}{sfx}"] = TensorSpec((rows, s.hidden))
            if s.qkv_bias:
                p[f"{prefix}{names[key]}{self._bias(names)}"] = TensorSpec((rows,))
        if self.row_eps is not None:
            p[f"{prefix}{names['q_norm']}{sfx}"] = TensorSpec((s.n_heads * self.dim,), init="ones_normal")
            p[f"{prefix}{names['k_norm']}{sfx}"] = TensorSpec((s.n_kv_heads * self.dim,), init="ones_normal")
        if self.v_mix == "mix":
            p[f"{prefix}{names['v_mix']}{sfx}"] = TensorSpec((), std=0.5)
        p[f"{prefix}{names['o']}{sfx}"] = TensorSpec((s.hidden, s.n_heads * self.vdim))
        if s.out_bias:
            p[f"{prefix}{names['o']}{self._bias(names)}"] = TensorSpec((s.hidden,))
        if self.has_sink:
            p[f"{prefix}{names['sink']}{sfx}"] = TensorSpec((s.n_heads,), std=1.0)
        return p

    @staticmethod
    def _bias(names: Dict[str, str]) -> str:
        return names.get("bias_suffix", ".bias")

    def _pieces(self):
        """(key, heads, size of a head) of the matrices that are stacked into the one projection, in its order of rows."""
        s = self.spec
        out = [("q", s.n_heads, self.dim)]
        if self.own_kv:
            out += [("k", s.n_kv_heads, self.dim), ("v", s.n_kv_heads, self.vdim)]
        if self.gated:
            out.append(("g", s.n_heads, self.vdim))
        return out

    def _pad_rows(self, t: torch.Tensor, heads: int, size: int) -> torch.Tensor:
        """[heads * size, K] -> [heads * hd, K]: every head's rows followed by zero rows up to the cache's head size."""
        if size == self.hd:
            return t
        out = torch.zeros((heads, self.hd, t.shape[1]), dtype=t.dtype, device=t.device)
        out[:, :size] = t.view(heads, size, t.shape[1])
        return out.view(heads * self.hd, t.shape[1])

    def load(self, tensors: Dict[str, torch.Tensor], prefix: str, names: Dict[str, str]) -> None:
        s = self.spec
        sfx = names.get("suffix", ".weight")
        bias = None
        if s.qkv_bias:
            bias = torch.cat([self._pad_rows(tensors[f"{prefix}{names[k]}{self._bias(names)}"].float()[:, None], heads, size)[:, 0]
                              for k, heads, size in self._pieces()])

        def rows(k, heads, size):
            t = tensors[f"{prefix}{names[k]}{sfx}"]
            if k in ("q", "k") and self.interleaved:
                t = t[self.position.to_half_split(heads, self.dim).to(t.device)]
            return self._pad_rows(t, heads, size)

        if self.interleaved and s.qkv_bias:
            raise ValueError("attention: neighbouring rotary pairs with biases on q and k are not implemented")
        self.qkv = Linear([rows(*piece) for piece in self._pieces()], bias, self.rt)
        if self.has_sink:
            self.sinks = self.rt.vector(tensors[f"{prefix}{names['sink']}{sfx}"])
        if self.row_eps is not None:                  # a head's padding is zero in q and k; its weights stay zero as well
            self.q_weight = self.rt.vector(self._pad_rows(tensors[f"{prefix}{names['q_norm']}{sfx}"].float()[:, None], s.n_heads, self.dim)[:, 0])
            self.k_weight = self.rt.vector(self._pad_rows(tensors[f"{prefix}{names['k_norm']}{sfx}"].float()[:, None], s.n_kv_heads, self.dim)[:, 0])
        if self.v_mix == "mix":
            self.mix = self.rt.vector(tensors[f"{prefix}{names['v_mix']}{sfx}"]).reshape(1)
        if self.slopes_host is not None:
            self.slopes = torch.tensor([float(m) for m in self.slopes_host], dtype=torch.float32, device=self.rt.device)
        ob = tensors[f"{prefix}{names['o']}{self._bias(names)}"] if s.out_bias else None
        wo = tensors[f"{prefix}{names['o']}{sfx}"]
        if self.vdim != self.hd:
            wo = self._pad_rows(wo.t().contiguous(), s.n_heads, self.vdim).t().contiguous()
        self.out = Linear(wo, ob, self.rt)

    def nbytes(self) -> int:
        return self.qkv.nbytes() + self.out.nbytes()

    def state(self, prefix: str, names: Dict[str, str]) -> Dict[str, torch.Tensor]:
        """The tensors of ``plan`` back out of the stacked matrices, as they are kept on the device."""
        out: Dict[str, torch.Tensor] = {}
        s, sfx = self.spec, names.get("suffix", ".weight")
        r = 0
        for key, heads, size in self._pieces():
            rows = heads * self.hd
            w = self.qkv.weight[r:r + rows]
            w = w if size == self.hd else w.view(heads, self.hd, -1)[:, :size].reshape(heads * size, -1)
            if key in ("q", "k") and self.interleaved:
                order = self.position.to_half_split(heads, size).to(w.device)
                back = torch.empty_like(w)
                back[order] = w
                w = back
            out[f"{prefix}{names[key]}{sfx}"] = w
            if self.qkv.bias is not None:
                b = self.qkv.bias[r:r + rows]
                out[f"{prefix}{names[key]}{self._bias(names)}"] = b if size == self.hd else b.view(heads, self.hd)[:, :size].reshape(-1)
            r += rows
        if self.row_eps is not None:
            out[f"{prefix}{names['q_norm']}{sfx}"] = self.q_weight.view(s.n_heads, self.hd)[:, :self.dim].reshape(-1)
            out[f"{prefix}{names['k_norm']}{sfx}"] = self.k_weight.view(s.n_kv_heads, self.hd)[:, :self.dim].reshape(-1)
        if self.v_mix == "mix":
            out[f"{prefix}{names['v_mix']}{sfx}"] = self.mix.reshape(())
        wo = self.out.weight
        out[f"{prefix}{names['o']}{sfx}"] = wo if self.vdim == self.hd else wo.view(-1, s.n_heads, self.hd)[:, :, :self.vdim].reshape(wo.shape[0], -1)
        if self.out.bias is not None:
            out[f"{prefix}{names['o']}{self._bias(names)}"] = self.out.bias
        if self.has_sink:
            out[f"{prefix}{names['sink']}{sfx}"] = self.sinks
        return out

    def scratch_row(self) -> int:
        """Values of the widest activation row a step of this part holds (its q | k | v row)."""
        return self.qd * (2 if self.gated else 1) + 2 * self.kvd

    graph_safe = True              # a decode step reads nothing of the batch on the host

    @property
    def short_context(self) -> int:
        """Positions up to which this mixer's decode kernel takes another road than for long contexts (none if 0):
        the stepper records decode steps for such contexts apart (``StepBatch.max_len`` is their bound)."""
        from ..kernels import short_context
        return short_context(self.hd)

    # ------------------------------------------------------------------ cache
    def cache_requests(self, site: int) -> List[object]:
        if self.spec.cache_from is not None:
            return []
        return [KVRequest(self.spec.n_kv_heads, self.hd, 0 if self.keep_first > 0 else self.spec.window)]

    # ------------------------------------------------------------------ step
    takes_pending_norm = True      # h may be a NormedInput: the q/k/v product folds the norm in when it can
    takes_next_norm = True         # forward(..., next_norm=): the norm that will read x next, for its last product

    def forward(self, h, x: torch.Tensor, batch, cache, site: int, next_norm=None):
        return self.out.accumulate(self._attend(h, batch, cache, site), x, next_norm)

    def produce(self, h, batch, cache, site: int) -> torch.Tensor:
        """The mixer's output as float32 rows of its own (what ``forward`` adds into x)."""
        return self.out.logits(self._attend(h, batch, cache, site))

    def _attend(self, h, batch, cache, site: int) -> torch.Tensor:
        s, K_ = self.spec, self.rt.kernels
        kv = cache.layer_kv(site)
        writes = s.cache_from is None
        rows = h.shape[0]
        if (not batch.prefill and writes and self.qkv._skinny(rows) and kv.storage.dtype is torch.bfloat16
                and self.position.rotary_dim == self.hd and self.amplitude == 1.0 and not self.qk_eps and not self.q_temp and not self.gated
                and self.row_eps is None and hasattr(K_, "qkv_rope")):
            # decoding: projection, rotation and the append to the cache as one kernel
            qkv = self.rt.empty(rows, self.qd + 2 * self.kvd)
            if self.qkv._folds(h, rows):
                K_.qkv_rope(h.xw, self.qkv.weight, self.qkv.bias, qkv, self.position.inv_freq, batch.row_pos,
                            batch.row_seq, batch.seq_slot, kv, s.n_heads, s.n_kv_heads, self.hd,
                            norm=(h.ssq, h.norm.spec.eps))
            else:
                K_.qkv_rope(h.tensor() if hasattr(h, "tensor") else h, self.qkv.weight, self.qkv.bias, qkv,
                            self.position.inv_freq, batch.row_pos, batch.row_seq, batch.seq_slot, kv, s.n_heads,
                            s.n_kv_heads, self.hd)
        elif self.row_eps is not None:
            qkv = self.qkv.store(h)
            mix = (self.mix, *batch.carried[FIRST_VALUES]) if self.v_mix == "mix" else None
            K_.row_norm_append(qkv, (self.q_weight, self.k_weight, self.dim, float(self.row_eps)), batch, kv, s.n_heads, s.n_kv_heads,
                               self.hd, self.vdim, mix)
            if self.v_mix == "first":                 # (the layer's own columns of its step's buffer, which nothing writes again)
                batch.carried[FIRST_VALUES] = (qkv[:, self.qd + self.kvd:], self.hd)
        else:
            qkv = self.qkv.store(h)
            opts = {}
            if self.amplitude != 1.0:
                opts["amplitude"] = self.amplitude
            if self.qk_eps:
                opts["qk_norm"] = (None, None, self.dim, float(self.qk_eps))
            if self.q_temp:
                opts["q_temp"] = self.q_temp
            K_.rope_append(qkv, self.position.inv_freq, self.position.rotary_dim, batch.row_pos, batch.row_seq,
                           batch.seq_slot, batch.seq_len, kv if writes else None, s.n_heads, self.nk, self.hd, **opts)
        att = self.rt.empty(h.shape[0], self.qd)
        from_cache = (not batch.prefill) or not writes
        more = {}
        if self.sink:
            more["sink"] = self.sink
        if self.keep_first:
            more["keep_first"] = self.keep_first
        if self.has_sink:
            more["head_sink"] = self.sinks
        if self.gated:
            more["gate_col"] = self.gate_col
        if self.slopes is not None:
            more["slopes"] = self.slopes
        K_.attention(qkv, kv, batch, att, s.n_heads, s.n_kv_heads, self.hd, s.scale, s.window, from_cache,
                     after_append=True, **more)
        return att


register_mixer("attention", Attention)
