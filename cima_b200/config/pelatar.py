"""Typed configuration of the Pelatar decoder, read from its own config.json keys.

A Pelatar model is a stack of layers whose norm stands on a sublayer's output only: x += N(mixer(x)); x += N(ff(x)), N an RMS
norm with a weight; the sublayers read the stream itself.  The head is the embedding table.

A layer's mixer is one of three kinds.  ``attention``: grouped-query softmax attention without rotation, q and k each divided
by their root mean square per head, the queries multiplied by a factor that grows with the position (``q_temp`` {coef,
every}), a stored number a head in the softmax's denominator, an output gate sigmoid(W_g h); with ``kv_from`` the layer reads
another layer's keys and values and stores no projections for them.  ``mlstm``: a matrix memory with exponential input and
forget gates and a running maximum.  ``gla``: linear attention with a decay per key channel.  The feed-forward is ``dense``
(gated, the tanh form of GELU), ``moe`` (softmax scores over experts and identity experts, a stored correction where groups
and experts are chosen, groups scored by their best expert, the chosen scores as weights), or absent (``mlp: null``).

config.json gives ``vocab``, ``width``, ``norm`` {eps} and per entry of ``layers``: ``type``, ``mixer`` and ``mlp``:
  attention   mixer {heads, kv_heads, dim, vdim, scale[, q_temp {coef, every}][, kv_from]}
  mlstm       mixer {heads, dim, vdim, gate_cap}
  gla         mixer {heads, dim, vdim, tau}
  mlp         {kind "dense", ff}  |  {kind "moe", expert {ff}, router {experts, top[, identity][, groups {count, keep}]}}
Tensor names: ``embed``, ``final.norm`` and under ``l<i>.``: ``norm1``, ``norm2``, ``mix.{q,k,v,g,o}`` with ``mix.sink``, or with
``mix.{norm,i,i.b,f,f.b}``, or with ``mix.{norm,a1,a2,a2.b}``, and ``mlp.{gate,up,down}`` or ``mlp.{router,correction,e<j>.{gate,up,
down}}``.  The rank of a1 / a2 stands in no key of a stored model: it is read off the tensors' shapes where a folder is given
(``from_dict(cfg, shapes)``); a configuration alone takes ``mixer.rank``, or 16.  Whether a model has sinks and corrections is
read off the stored names in the same way.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .qwen2 import ConfigError
from .specs import BlockSpec, FeedForwardSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec
from .vunovik import _int, _num

MAX_POSITION = 1 << 20       # nothing in the design ends at a position
DEFAULT_RANK = 16


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[Tuple[float, int]]         # coef, every
    sink: bool
    kv_from: Optional[int]


@dataclass(frozen=True)
class MemoryMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float = 0.0                       # mlstm
    tau: float = 0.0                            # gla
    rank: int = 0                               # gla


@dataclass(frozen=True)
class Experts:
    experts: int
    identity: int
    top: int
    ff: int
    groups: int
    keep: int
    correction: bool


@dataclass(frozen=True)
class PelatarLayer:
    kind: str                                   # "attention" | "mlstm" | "gla"
    attention: Optional[AttentionMixer] = None
    memory: Optional[MemoryMixer] = None
    dense_ff: int = 0                           # > 0: the dense feed-forward's middle
    moe: Optional[Experts] = None


def _has(shapes, name: str, default: bool) -> bool:
    return default if shapes is None else name in shapes


def _positive(d: Dict[str, Any], key: str, where: str) -> float:
    v = _num(d, key, where)
    if v <= 0:
        raise ConfigError(f"config.json: {where}{key} ({v}) must be positive")
    return v


def _attention(m: Dict[str, Any], where: str, sink: bool) -> AttentionMixer:
    dim, heads = _int(m, "dim", where), _int(m, "heads", where)
    temp = m.get("q_temp")
    a = AttentionMixer(heads=heads, kv_heads=_int(m, "kv_heads", where) if m.get("kv_heads") is not None else heads, dim=dim,
                       vdim=_int(m, "vdim", where) if m.get("vdim") is not None else dim,
                       scale=_num(m, "scale", where) if m.get("scale") is not None else dim ** -0.5,
                       q_temp=(_num(temp, "coef", where + "q_temp."), _int(temp, "every", where + "q_temp.")) if temp is not None else None,
                       sink=sink, kv_from=_int(m, "kv_from", where, least=0) if m.get("kv_from") is not None else None)
    if a.heads % a.kv_heads:
        raise ConfigError(f"config.json: {where}heads ({a.heads}) must be a multiple of kv_heads ({a.kv_heads})")
    return a


def _experts(f: Dict[str, Any], where: str, correction: bool) -> Experts:
    r, e = f.get("router"), f.get("expert")
    n = _int(r, "experts", where + "router.")
    identity = _int(r, "identity", where + "router.", least=0) if r.get("identity") is not None else 0
    g = r.get("groups")
    groups = _int(g, "count", where + "router.groups.") if g is not None else 1
    keep = _int(g, "keep", where + "router.groups.") if g is not None else 1
    top = _int(r, "top", where + "router.")
    if (n + identity) % groups or keep > groups:
        raise ConfigError(f"config.json: {where}router.groups: {groups} groups of which {keep} stay do not fit {n} + {identity} experts")
    if top > keep * ((n + identity) // groups):
        raise ConfigError(f"config.json: {where}router.top ({top}) exceeds the experts that stay ({keep * ((n + identity) // groups)})")
    return Experts(experts=n, identity=identity, top=top, ff=_int(e, "ff", where + "expert."), groups=groups, keep=keep, correction=correction)


@dataclass(frozen=True)
class PelatarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[PelatarLayer, ...]

    ARCHITECTURE = "Pelatar"

    @classmethod
    def from_dict(cls, cfg: Dict[str, Any], shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> "PelatarConfig":
        if cfg.get("architecture") != cls.ARCHITECTURE:
            raise ConfigError(f"config.json: architecture {cfg.get('architecture')!r} is not '{cls.ARCHITECTURE}'")
        vocab, width = _int(cfg, "vocab", ""), _int(cfg, "width", "")
        eps = _positive(cfg.get("norm"), "eps", "norm.")
        raw_layers = cfg.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]."
            kind = L.get("type") if isinstance(L, dict) else None
            m = L.get("mixer") if isinstance(L, dict) else None
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: {where}mixer is missing")
            dense_ff, moe = 0, None
            f = L.get("mlp")
            if f is not None:
                if not isinstance(f, dict) or f.get("kind") not in ("dense", "moe"):
                    raise ConfigError(f"config.json: {where}mlp.kind {f.get('kind') if isinstance(f, dict) else f!r} is neither 'dense' nor 'moe'")
                if f["kind"] == "dense":
                    dense_ff = _int(f, "ff", where + "mlp.")
                else:
                    if not isinstance(f.get("router"), dict):
                        raise ConfigError(f"config.json: {where}mlp.router is missing")
                    moe = _experts(f, where + "mlp.", _has(shapes, f"l{i}.mlp.correction", True))
            wm = where + "mixer."
            if kind == "attention":
                a = _attention(m, wm, _has(shapes, f"l{i}.mix.sink", True))
                if a.kv_from is not None:
                    src = layers[a.kv_from].attention if a.kv_from < i else None
                    if src is None or src.kv_from is not None:
                        raise ConfigError(f"config.json: {wm}kv_from ({a.kv_from}) must name an earlier attention layer with keys and "
                                          f"values of its own")
                    if (src.kv_heads, src.dim, src.vdim) != (a.kv_heads, a.dim, a.vdim):
                        raise ConfigError(f"config.json: {wm}kv_from: layer {a.kv_from} differs in kv_heads, dim or vdim")
                layers.append(PelatarLayer(kind=kind, attention=a, dense_ff=dense_ff, moe=moe))
            elif kind in ("mlstm", "gla"):
                sizes = dict(heads=_int(m, "heads", wm), dim=_int(m, "dim", wm),
                             vdim=_int(m, "vdim", wm) if m.get("vdim") is not None else _int(m, "dim", wm))
                if kind == "mlstm":
                    mem = MemoryMixer(gate_cap=_positive(m, "gate_cap", wm), **sizes)
                else:
                    rank = _int(m, "rank", wm) if m.get("rank") is not None else DEFAULT_RANK
                    if shapes is not None and f"l{i}.mix.a1" in shapes:
                        rank = int(shapes[f"l{i}.mix.a1"][0])
                    mem = MemoryMixer(tau=_positive(m, "tau", wm), rank=rank, **sizes)
                layers.append(PelatarLayer(kind=kind, memory=mem, dense_ff=dense_ff, moe=moe))
            else:
                raise ConfigError(f"config.json: {where}type {kind!r} is none of 'attention', 'mlstm', 'gla'")
        return cls(vocab=vocab, width=width, norm_eps=eps, layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        out = []
        for L in self.layers:
            if L.kind == "attention":
                a = L.attention
                mixer: Dict[str, Any] = {"dim": a.dim, "heads": a.heads, "kv_heads": a.kv_heads, "scale": a.scale, "vdim": a.vdim}
                if a.q_temp is not None:
                    mixer["q_temp"] = {"coef": a.q_temp[0], "every": a.q_temp[1]}
                if a.kv_from is not None:
                    mixer["kv_from"] = a.kv_from
            else:
                g = L.memory
                mixer = {"dim": g.dim, "heads": g.heads, "vdim": g.vdim}
                mixer.update({"gate_cap": g.gate_cap} if L.kind == "mlstm" else {"rank": g.rank, "tau": g.tau})
            mlp: Optional[Dict[str, Any]] = None
            if L.dense_ff:
                mlp = {"ff": L.dense_ff, "kind": "dense"}
            elif L.moe is not None:
                e = L.moe
                mlp = {"expert": {"ff": e.ff}, "kind": "moe", "router": {"experts": e.experts, "groups": {"count": e.groups, "keep": e.keep},
                                                                          "identity": e.identity, "top": e.top}}
            out.append({"mixer": mixer, "mlp": mlp, "type": L.kind})
        return {"architecture": self.ARCHITECTURE, "layers": out, "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = NormSpec(kind="rmsnorm", size=W, eps=eps)
        blocks = []
        for i, L in enumerate(self.layers):
            names = {"mixer_norm": "norm1", "ffn_norm": "norm2", "gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down", "experts": "mlp.",
                     "suffix": ""}
            names.update({k: f"mix.{k}" for k in ("q", "k", "v", "g", "o")})
            if L.kind == "attention":
                a = L.attention
                params: Dict[str, Any] = {"v_dim": a.vdim, "qk_norm_eps": eps, "head_sink": a.sink, "gate": True, "own_kv": a.kv_from is None}
                if a.q_temp is not None:
                    params["q_temp"] = a.q_temp
                mixer = MixerSpec(kind="attention", hidden=W, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim, scale=a.scale,
                                  position=PositionSpec(kind="none", head_dim=a.dim, rotary_dim=0, theta=0.0), cache_from=a.kv_from,
                                  params=params)
                names["sink"] = "mix.sink"
            else:
                g = L.memory
                params = {"v_dim": g.vdim, "eps": eps}
                names["norm"] = "mix.norm"
                if L.kind == "mlstm":
                    params["gate_cap"] = g.gate_cap
                    names.update({"i": "mix.i", "f": "mix.f", "i_bias": "mix.i.b", "f_bias": "mix.f.b"})
                else:
                    params.update({"tau": g.tau, "rank": g.rank})
                    names.update({"a1": "mix.a1", "a2": "mix.a2", "a2_bias": "mix.a2.b"})
                mixer = MixerSpec(kind="mlstm" if L.kind == "mlstm" else "gated_linear_attention", hidden=W, n_heads=g.heads,
                                  n_kv_heads=g.heads, head_dim=g.dim, params=params)
            ffn = None
            if L.dense_ff:
                ffn = FeedForwardSpec(kind="gated_mlp", hidden=W, intermediate=L.dense_ff, activation="gelu_tanh")
            elif L.moe is not None:
                e = L.moe
                ffn = FeedForwardSpec(kind="moe", hidden=W, intermediate=e.ff, activation="silu",
                                      params={"experts": e.experts, "identity": e.identity, "top": e.top, "groups": e.groups, "keep": e.keep,
                                              "scoring": "softmax", "correction": e.correction, "group_score": "best", "normalize": False})
            blocks.append(BlockSpec(kind="branchnorm", mixer=mixer, feed_forward=ffn, mixer_norm=norm,
                                    ffn_norm=norm if ffn is not None else None, prefix=f"l{i}.", names=names))
        return ModelSpec(architecture=self.ARCHITECTURE, vocab=self.vocab, hidden=W, max_position=MAX_POSITION, layers=blocks,
                         schedule=list(range(len(blocks))), final_norm=norm, tie_head=True, embed_name="embed",
                         final_norm_name="final.norm", head_name="head")
