"""Typed configuration of the Gudarax decoder, read from its own config.json keys.

A Gudarax model is a stack of pre-norm layers (RMS norms with plain weights); behind its feed-forward every layer adds a
*token input*: a slice of a side table's row for the token, gated by a small projection of the stream, projected to the
model's width and RMS-normed.  A learned vector a position is added to the scaled embedding; the head is a matrix of its own.

A layer's mixer is one of three kinds.  ``latent_attention``: attention over latents without positions, the queries through a
latent of their own, an output gate sigmoid(W_g h).  ``delta``: the gated delta rule with one decay a head, short causal
convolutions on q, k and v, and a SiLU gate behind the heads' norm.  ``attention``: grouped-query softmax attention with biases
on q, k and v, an RMS norm over the whole q and the whole k projection, a distance bias -2^(-8 (h + 1) / H) (i - j) instead of
a rotation, behind a window; with ``v_mix`` a layer's values are mixed with those of the first such layer.  The feed-forward is
``dense`` (gated, SiLU), ``moe`` (sigmoid scores, unnormalised weights that multiply an expert's input, ungated experts with
the square of ReLU), or absent (``mlp: null``).

config.json gives ``vocab``, ``width``, ``max_positions``, ``norm`` {eps}, ``embedding`` {scale}, ``token_side`` {dim} and per
entry of ``layers``: ``type``, ``mixer`` and ``mlp``:
  latent_attention  mixer {heads, dim, vdim, kv_rank, q_rank, scale}
  delta             mixer {heads, kv_heads, dim, vdim, conv}
  attention         mixer {heads, kv_heads, dim, vdim, scale[, mask {size}][, v_mix]}
  mlp               {kind "dense", ff}  |  {kind "moe", expert {ff}, router {experts, top}}
Tensor names: ``embed``, ``pos``, ``side.embed``, ``final.norm``, ``head`` and under ``l<i>.``: ``norm1``, ``norm2``,
``side.{gate,proj,norm}``, ``mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,g,o}``, or ``mix.{q,k,v}`` with ``.conv`` and
``mix.{b,a,A_log,dt_bias,norm,g,o}``, or ``mix.{q,k,v}`` with ``.b``, ``mix.{q.norm,k.norm,vmix,o}``, and
``mlp.{gate,up,down}`` or ``mlp.{router,e<j>.{up,down}}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .qwen2 import ConfigError
from .specs import BlockSpec, FeedForwardSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, TokenSideSpec
from .vunovik import _int, _num


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                                 # 0 = every earlier position
    v_mix: bool


@dataclass(frozen=True)
class GudaraxLayer:
    kind: str                                   # "latent_attention" | "delta" | "attention"
    latent: Optional[LatentMixer] = None
    delta: Optional[DeltaMixer] = None
    attention: Optional[AttentionMixer] = None
    dense_ff: int = 0                           # > 0: the dense feed-forward's middle
    moe: Optional[Tuple[int, int, int]] = None  # experts, top, ff


def _positive(d: Any, key: str, where: str) -> float:
    v = _num(d, key, where)
    if v <= 0:
        raise ConfigError(f"config.json: {where}{key} ({v}) must be positive")
    return v


def _or(d: Dict[str, Any], key: str, where: str, default: int) -> int:
    return _int(d, key, where) if d.get(key) is not None else default


def _mixer(kind: Any, m: Dict[str, Any], where: str):
    heads, dim = _int(m, "heads", where), _int(m, "dim", where)
    vdim = _or(m, "vdim", where, dim)
    scale = _positive(m, "scale", where) if m.get("scale") is not None else dim ** -0.5
    if kind == "latent_attention":
        return LatentMixer(heads=heads, dim=dim, vdim=vdim, kv_rank=_int(m, "kv_rank", where), q_rank=_int(m, "q_rank", where), scale=scale)
    kv_heads = _or(m, "kv_heads", where, heads)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    if kind == "delta":
        return DeltaMixer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=_int(m, "conv", where))
    mask = m.get("mask")
    window = _int(mask, "size", where + "mask.", least=0) if mask is not None and mask.get("size") is not None else 0
    return AttentionMixer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, window=window, v_mix=bool(m.get("v_mix", False)))


@dataclass(frozen=True)
class GudaraxConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    embedding_scale: float
    side_dim: int
    layers: Tuple[GudaraxLayer, ...]

    ARCHITECTURE = "Gudarax"
    KINDS = {"latent_attention": "latent", "delta": "delta", "attention": "attention"}

    @classmethod
    def from_dict(cls, cfg: Dict[str, Any]) -> "GudaraxConfig":
        if cfg.get("architecture") != cls.ARCHITECTURE:
            raise ConfigError(f"config.json: architecture {cfg.get('architecture')!r} is not '{cls.ARCHITECTURE}'")
        vocab, width, positions = _int(cfg, "vocab", ""), _int(cfg, "width", ""), _int(cfg, "max_positions", "")
        eps = _positive(cfg.get("norm"), "eps", "norm.")
        scale = _num(cfg["embedding"], "scale", "embedding.") if cfg.get("embedding") is not None else 1.0
        side = _int(cfg.get("token_side"), "dim", "token_side.")
        raw_layers = cfg.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]."
            kind = L.get("type") if isinstance(L, dict) else None
            if kind not in cls.KINDS:
                raise ConfigError(f"config.json: {where}type {kind!r} is none of {sorted(cls.KINDS)}")
            if not isinstance(L.get("mixer"), dict):
                raise ConfigError(f"config.json: {where}mixer is missing")
            dense_ff, moe = 0, None
            f = L.get("mlp")
            if f is not None:
                if not isinstance(f, dict) or f.get("kind") not in ("dense", "moe"):
                    raise ConfigError(f"config.json: {where}mlp.kind {f.get('kind') if isinstance(f, dict) else f!r} is neither 'dense' nor 'moe'")
                if f["kind"] == "dense":
                    dense_ff = _int(f, "ff", where + "mlp.")
                else:
                    r = f.get("router")
                    moe = (_int(r, "experts", where + "mlp.router."), _int(r, "top", where + "mlp.router."), _int(f.get("expert"), "ff", where + "mlp.expert."))
                    if moe[1] > moe[0]:
                        raise ConfigError(f"config.json: {where}mlp.router.top ({moe[1]}) exceeds its experts ({moe[0]})")
            layers.append(GudaraxLayer(kind=kind, dense_ff=dense_ff, moe=moe, **{cls.KINDS[kind]: _mixer(kind, L["mixer"], where + "mixer.")}))
        mixing = [(i, L.attention) for i, L in enumerate(layers) if L.attention is not None and L.attention.v_mix]
        for i, a in mixing[1:]:
            if (a.kv_heads, a.vdim) != (mixing[0][1].kv_heads, mixing[0][1].vdim):
                raise ConfigError(f"config.json: layers[{i}].mixer.v_mix: layer {mixing[0][0]}, whose values are mixed in, differs in kv_heads or vdim")
        return cls(vocab=vocab, width=width, max_positions=positions, norm_eps=eps, embedding_scale=scale, side_dim=side, layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        out = []
        for L in self.layers:
            if L.kind == "latent_attention":
                a = L.latent
                mixer: Dict[str, Any] = {"dim": a.dim, "heads": a.heads, "kv_rank": a.kv_rank, "q_rank": a.q_rank, "scale": a.scale, "vdim": a.vdim}
            elif L.kind == "delta":
                d = L.delta
                mixer = {"conv": d.conv, "dim": d.dim, "heads": d.heads, "kv_heads": d.kv_heads, "vdim": d.vdim}
            else:
                g = L.attention
                mixer = {"dim": g.dim, "heads": g.heads, "kv_heads": g.kv_heads, "scale": g.scale, "v_mix": g.v_mix, "vdim": g.vdim}
                if g.window:
                    mixer["mask"] = {"size": g.window}
            mlp: Optional[Dict[str, Any]] = None
            if L.dense_ff:
                mlp = {"ff": L.dense_ff, "kind": "dense"}
            elif L.moe is not None:
                mlp = {"expert": {"ff": L.moe[2]}, "kind": "moe", "router": {"experts": L.moe[0], "top": L.moe[1]}}
            out.append({"mixer": mixer, "mlp": mlp, "type": L.kind})
        return {"architecture": self.ARCHITECTURE, "embedding": {"scale": self.embedding_scale}, "layers": out,
                "max_positions": self.max_positions, "norm": {"eps": self.norm_eps}, "token_side": {"dim": self.side_dim},
                "vocab": self.vocab, "width": self.width}

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = NormSpec(kind="rmsnorm", size=W, eps=eps)
        side = TokenSideSpec(name="side.embed", dim=self.side_dim, eps=eps, activation="gelu_tanh")
        blocks = []
        first_mix = True
        for i, L in enumerate(self.layers):
            names = {"mixer_norm": "norm1", "ffn_norm": "norm2", "gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down", "experts": "mlp.",
                     "side_gate": "side.gate", "side_proj": "side.proj", "side_norm": "side.norm", "suffix": "", "bias_suffix": ".b"}
            if L.kind == "latent_attention":
                a = L.latent
                mixer = MixerSpec(kind="latent_attention", hidden=W, n_heads=a.heads, n_kv_heads=1, head_dim=a.dim, scale=a.scale,
                                  params={"v_dim": a.vdim, "kv_rank": a.kv_rank, "q_rank": a.q_rank, "latent_eps": eps, "gate": True})
                names.update({"q_down": "mix.dq", "q_norm": "mix.dq.norm", "q": "mix.uq", "latent": "mix.dkv", "latent_norm": "mix.dkv.norm",
                              "k_up": "mix.uk", "v_up": "mix.uv", "g": "mix.g", "o": "mix.o"})
            elif L.kind == "delta":
                d = L.delta
                mixer = MixerSpec(kind="delta", hidden=W, n_heads=d.heads, n_kv_heads=d.kv_heads, head_dim=d.dim,
                                  params={"v_dim": d.vdim, "taps": d.conv, "eps": eps})
                names.update({k: f"mix.{k}" for k in ("q", "k", "v", "b", "a", "A_log", "dt_bias", "norm", "g", "o")})
            else:
                g = L.attention
                params: Dict[str, Any] = {"v_dim": g.vdim, "row_norm_eps": eps,
                                          "distance_slopes": [2.0 ** (-8.0 * (h + 1) / g.heads) for h in range(g.heads)]}
                if g.v_mix:
                    params["v_mix"] = "first" if first_mix else "mix"
                    first_mix = False
                mixer = MixerSpec(kind="attention", hidden=W, n_heads=g.heads, n_kv_heads=g.kv_heads, head_dim=g.dim, scale=g.scale,
                                  window=g.window, qkv_bias=True, params=params,
                                  position=PositionSpec(kind="none", head_dim=g.dim, rotary_dim=0, theta=0.0))
                names.update({k: f"mix.{k}" for k in ("q", "k", "v", "o")})
                names.update({"q_norm": "mix.q.norm", "k_norm": "mix.k.norm", "v_mix": "mix.vmix"})
            ffn = None
            if L.dense_ff:
                ffn = FeedForwardSpec(kind="gated_mlp", hidden=W, intermediate=L.dense_ff, activation="silu")
            elif L.moe is not None:
                experts, top, ff = L.moe
                ffn = FeedForwardSpec(kind="moe", hidden=W, intermediate=ff, activation="relu2",
                                      params={"experts": experts, "top": top, "normalize": False, "gated": False, "weight_on": "input"})
            blocks.append(BlockSpec(kind="prenorm", mixer=mixer, feed_forward=ffn, mixer_norm=norm, ffn_norm=norm if ffn is not None else None,
                                    prefix=f"l{i}.", names=names, token_side=side))
        return ModelSpec(architecture=self.ARCHITECTURE, vocab=self.vocab, hidden=W, max_position=self.max_positions, layers=blocks,
                         schedule=list(range(len(blocks))), final_norm=norm, tie_head=False, embed_name="embed",
                         final_norm_name="final.norm", head_name="head", embed_scale=self.embedding_scale, embed_positions="pos",
                         token_side=side, unread=("l*.norm2", "l*.mix.vmix"))
