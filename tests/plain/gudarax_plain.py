"""Plain, slow implementation of the Gudarax decoder: the oracle of its tests.

Whole sequences, no cache, no batching, one function per mechanism, float64 by default.  It shares no code
with the ``cima_b200`` package: the configuration is a plain dict with config.json's own keys, the weights a
plain dict name -> tensor (``read_folder`` reads both from a model folder with nothing but the standard library
and torch).

The design in this file's notation (T tokens of one sequence, width W, t a position counted from 0):

  x_t  = s E[tok_t] + P[t];   rms(z) = z / sqrt(mean(z^2) + eps)
  x   <- x + mixer(rms(x) w1);   x <- x + ff(rms(x) w2)        (second line only where the layer has a feed-forward)
  x   <- x + rms(V (gelu_tanh(U x) * D_i[tok])) w3             D_i[tok]: layer i's part of the token's row of a side table
  logits = H (rms(x) w_f)

  "latent_attention":  q = W_uq (rms(W_dq h) w_q);  c = rms(W_dkv h) w_c;  keys W_uk c and values W_uv c, head by head;
        softmax over all earlier positions of q . k * scale;  heads concatenated times sigmoid(W_g h), then W_o
  "delta":  q, k, v = silu(taps(W h)) per channel over time;  q, k to unit length per head, q also times dim^(-1/2);
        beta = sigmoid(W_b h);  g = exp(-exp(A) softplus(W_a h + d)), one of each a head;
        S' = g S + k (beta (v - g S^T k))^T, read out as o = S'^T q;  rms(o) w per head times silu(W_g h), then W_o
  "attention":  q, k, v = W h + b;  q and k each rms-normed over all their heads at once, with a weight;
        score(i, j) = q_i . k_j * scale - m_h (i - j), m_h = 2^(-8 (h + 1) / H);  j within the window;
        v <- (1 - l) v + l v1 in every mixing layer but the first, v1 the first one's values;  then W_o
  "dense":  W_d (silu(W_g h) * W_u h)
  "moe":  s = sigmoid(W_r h); the top largest; y = sum_e W_d relu(W_u (s_e h))^2
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch


# ---------------------------------------------------------------------------------------------- files
def read_folder(folder: str, dtype=torch.float64):
    """(config dict, {name: tensor}) of a model folder; floating tensors in ``dtype``, integer ones as they are."""
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "F64": torch.float64, "I32": torch.int32,
             "I64": torch.int64}
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        t = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[info["dtype"]]).reshape(info["shape"])
        out[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, out


# ---------------------------------------------------------------------------------------------- small pieces
def plain_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def plain_silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def plain_gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def plain_embedding(ids, table, positions, scale: float) -> torch.Tensor:
    return torch.stack([table[int(tok)] * scale + positions[t] for t, tok in enumerate(ids)])


def plain_slopes(heads: int):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def plain_visible(t: int, window: int):
    """Positions that position t sees: all up to itself, or with a window the last ``window`` of them."""
    return list(range(max(0, t - window + 1) if window else 0, t + 1))


def plain_taps(z: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """z [T, C], w [C, taps]: y_t = sum_j w[:, j] z_(t - taps + 1 + j), zeros before the start."""
    out = torch.zeros_like(z)
    taps = w.shape[1]
    for j in range(taps):
        back = taps - 1 - j
        if back < z.shape[0]:
            out[back:] += w[:, j] * z[:z.shape[0] - back]
    return out


# ---------------------------------------------------------------------------------------------- mixers
def plain_latent_attention(h, W, m: dict, eps: float, weights_out=None):
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = ((plain_rms(h @ W["dq"].T, eps) * W["dq.norm"]) @ W["uq"].T).reshape(T, H, dim)
    c = plain_rms(h @ W["dkv"].T, eps) * W["dkv.norm"]
    k, v = (c @ W["uk"].T).reshape(T, H, dim), (c @ W["uv"].T).reshape(T, H, vdim)
    P = torch.zeros((H, T, T), dtype=h.dtype)
    out = torch.zeros((T, H, vdim), dtype=h.dtype)
    for a in range(H):
        s = (q[:, a] @ k[:, a].T) * m["scale"]
        for t in range(T):
            P[a, t, :t + 1] = torch.softmax(s[t, :t + 1], dim=0)
        out[:, a] = P[a] @ v[:, a]
    if weights_out is not None:
        weights_out.append(P)
    return (out.reshape(T, H * vdim) * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


def plain_mixed_values(v, first, lam: float):
    """What a mixing layer uses of its own values and the first mixing layer's (None: this is the first)."""
    return v if first is None else (1.0 - lam) * v + lam * first


def plain_attention(h, W, m: dict, eps: float, first_values=None, weights_out=None):
    """(the mixer's output, its own values [T, kv_heads * vdim] before any mixing)."""
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    window = (m.get("mask") or {}).get("size", 0)
    q = (plain_rms(h @ W["q"].T + W["q.b"], eps) * W["q.norm"]).reshape(T, H, dim)
    k = (plain_rms(h @ W["k"].T + W["k.b"], eps) * W["k.norm"]).reshape(T, G, dim)
    own = h @ W["v"].T + W["v.b"]
    v = (plain_mixed_values(own, first_values, W.get("vmix")) if m.get("v_mix") else own).reshape(T, G, vdim)
    P = torch.zeros((H, T, T), dtype=h.dtype)
    out = torch.zeros((T, H, vdim), dtype=h.dtype)
    for a, slope in enumerate(plain_slopes(H)):
        g = a // (H // G)
        for t in range(T):
            seen = plain_visible(t, window)
            dist = torch.tensor([float(t - j) for j in seen], dtype=h.dtype)
            P[a, t, seen] = torch.softmax((k[seen, g] @ q[t, a]) * m["scale"] - slope * dist, dim=0)
        out[:, a] = P[a] @ v[:, g]
    if weights_out is not None:
        weights_out.append(P)
    return out.reshape(T, H * vdim) @ W["o"].T, own


def plain_delta_inputs(h, W, m: dict):
    """(q, k [T, kv_heads, dim], v [T, heads, vdim], beta, g [T, heads]) as the rule takes them."""
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (plain_silu(plain_taps(h @ W[n].T, W[n + ".conv"])) for n in ("q", "k", "v"))
    q, k = q.reshape(T, G, dim), k.reshape(T, G, dim)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * dim ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    z = h @ W["a"].T + W["dt_bias"]
    softplus = torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))
    return q, k, v.reshape(T, H, vdim), torch.sigmoid(h @ W["b"].T), torch.exp(-torch.exp(W["A_log"]) * softplus)


def plain_delta_rule(q, k, v, beta, g):
    """One token after another; o [T, heads, vdim]."""
    T, H, vdim = v.shape
    share = H // q.shape[1]
    out = torch.zeros_like(v)
    for a in range(H):
        S = torch.zeros((q.shape[2], vdim), dtype=v.dtype)
        for t in range(T):
            kt, qt = k[t, a // share], q[t, a // share]
            S = g[t, a] * S
            S = S + torch.outer(kt, beta[t, a] * (v[t, a] - S.T @ kt))
            out[t, a] = S.T @ qt
    return out


def plain_delta(h, W, m: dict, eps: float):
    T = h.shape[0]
    o = plain_rms(plain_delta_rule(*plain_delta_inputs(h, W, m)), eps) * W["norm"]
    return (o.reshape(T, -1) * plain_silu(h @ W["g"].T)) @ W["o"].T


# ---------------------------------------------------------------------------------------------- feed-forwards, side input
def plain_dense_ff(h, W):
    return (plain_silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def plain_route(s: torch.Tensor, top: int):
    """Scores of one token -> the chosen experts."""
    return sorted(range(s.numel()), key=lambda e: -float(s[e]))[:top]


def plain_moe(h, W, router: dict):
    s = torch.sigmoid(h @ W["router"].T)
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in plain_route(s[t], router["top"]):
            z = torch.clamp(W[f"e{e}.up"] @ (s[t, e] * h[t]), min=0.0)
            y[t] += W[f"e{e}.down"] @ (z * z)
    return y


def plain_side_input(x, ids, table, layer: int, dim: int, W, eps: float):
    """What layer ``layer``'s token input adds to the stream."""
    e = table[torch.as_tensor(ids, dtype=torch.long)][:, layer * dim:(layer + 1) * dim]
    y = (plain_gelu_tanh(x @ W["gate"].T) * e) @ W["proj"].T
    return plain_rms(y, eps) * W["norm"]


# ---------------------------------------------------------------------------------------------- the model
def _sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def plain_forward(cfg: dict, weights: dict, ids, return_layers: bool = False, attention_out=None):
    """Logits [T, vocab] of one sequence (and the stream after every layer).  ``attention_out``: a dict that receives the
    softmax weights of every attention layer by its index."""
    eps = cfg["norm"]["eps"]
    x = plain_embedding(ids, weights["embed"], weights["pos"], cfg["embedding"]["scale"])
    streams, first_values = [], None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m, W, seen = layer["mixer"], _sub(weights, p + "mix."), []
        h = plain_rms(x, eps) * weights[p + "norm1"]
        if layer["type"] == "latent_attention":
            y = plain_latent_attention(h, W, m, eps, seen)
        elif layer["type"] == "delta":
            y = plain_delta(h, W, m, eps)
        elif layer["type"] == "attention":
            y, own = plain_attention(h, W, m, eps, first_values, seen)
            if m.get("v_mix") and first_values is None:
                first_values = own
        else:
            raise ValueError(f"unknown layer type {layer['type']!r}")
        if attention_out is not None and seen:
            attention_out[i] = seen[0]
        x = x + y
        mlp = layer.get("mlp")
        if mlp is not None:
            h, W = plain_rms(x, eps) * weights[p + "norm2"], _sub(weights, p + "mlp.")
            x = x + (plain_dense_ff(h, W) if mlp["kind"] == "dense" else plain_moe(h, W, mlp["router"]))
        x = x + plain_side_input(x, ids, weights["side.embed"], i, cfg["token_side"]["dim"], _sub(weights, p + "side."), eps)
        streams.append(x)
    logits = (plain_rms(x, eps) * weights["final.norm"]) @ weights["head"].T
    return (logits, torch.stack(streams)) if return_layers else logits
