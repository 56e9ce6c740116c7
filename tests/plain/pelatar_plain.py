"""Plain, slow implementation of the Pelatar decoder: the oracle of its tests.

Whole sequences, no cache, no batching, one function per mechanism, float64 by default.  It shares no code
with the ``cima_b200`` package: the configuration is a plain dict with config.json's own keys, the weights a
plain dict name -> tensor (``read_folder`` reads both from a model folder with nothing but the standard library
and torch).

The design in this file's notation (T tokens of one sequence, width W, t a position counted from 0):

  x_t  = E[tok_t];   rms(z) = z / sqrt(mean(z^2) + eps)
  x   <- x + w1 * rms(mixer(x));   x <- x + w2 * rms(ff(x))    (second line only where the layer has a feed-forward)
  logits = E (w_f * rms(x))

  "attention":  grouped heads; q, k <- rms(q), rms(k) per head over its own values; q_t also times
        1 + coef ln(floor((t + 1) / every) + 1); scores q . k * scale; every earlier position is seen; the softmax's
        denominator holds exp(sink_h) besides; heads concatenated, times sigmoid(W_g x) value by value, then W_o.
        A layer with ``kv_from`` j takes layer j's finished keys and values instead of making its own.
  "mlstm":  q = W_q x / sqrt(dim), k = W_k x, v = W_v x;  i = cap tanh((W_i x + b_i) / cap),
        f = -log(1 + exp(-cap tanh((W_f x + b_f) / cap))), one of each a head;
        m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' = e^(f + m - m') n + e^(i - m') k;
        o = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6);  m, S, n start at 0;
        rms(o) per head, all heads times one weight vector, times sigmoid(W_g x), then W_o
  "gla":  q = W_q x / sqrt(dim), k = W_k x, v = W_v x;  a = sigmoid(W_a2 W_a1 x + b)^(1 / tau) per head and key channel;
        S' = diag(a) S + k v^T;  o = S'^T q;  rms(o) per head times a weight all heads share, times silu(W_g x), then W_o
  "dense":  W_d (gelu_tanh(W_g x) * W_u x)
  "moe":  s = softmax(W_r x) over experts and identity experts; c = s + correction; equal groups of neighbours, a group's
        score its largest c, the best ``keep`` groups stay; the ``top`` largest c among them are chosen, each weighted with
        its s as it is; an expert is W_d (silu(W_g x) * W_u x), an identity expert (the last ones) is x
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


def plain_gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def plain_silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def plain_log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    """log(1 / (1 + e^(-z))), written so that neither tail overflows."""
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def plain_query_temperature(position: int, coef: float, every: int) -> float:
    return 1.0 + coef * math.log((position + 1) // every + 1)


def plain_sink_softmax(scores: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """softmax of a row of scores whose denominator also holds exp(sink): the weights sum to less than 1."""
    top = max(float(scores.max()), float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum() + math.exp(float(sink) - top))


# ---------------------------------------------------------------------------------------------- mixers
def plain_keys_values(h, W, m: dict, eps: float):
    """A layer's finished keys [T, kv_heads, dim] (normed) and values [T, kv_heads, vdim]."""
    T, G = h.shape[0], m["kv_heads"]
    return plain_rms((h @ W["k"].T).reshape(T, G, m["dim"]), eps), (h @ W["v"].T).reshape(T, G, m["vdim"])


def plain_attention(h, W, m: dict, eps: float, keys_values=None, weights_out=None):
    """The softmax mixer; ``keys_values`` (another layer's, from ``plain_keys_values``) where the layer has none of its
    own.  ``weights_out``: a list that receives [heads, T, T], the softmax weights."""
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = plain_rms((h @ W["q"].T).reshape(T, H, dim), eps)
    temp = m.get("q_temp")
    if temp:
        q = q * torch.tensor([plain_query_temperature(t, temp["coef"], temp["every"]) for t in range(T)], dtype=h.dtype)[:, None, None]
    k, v = keys_values if keys_values is not None else plain_keys_values(h, W, m, eps)
    out = torch.zeros((T, H, vdim), dtype=h.dtype)
    P = torch.zeros((H, T, T), dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        for i in range(T):
            P[a, i, :i + 1] = plain_sink_softmax((k[:i + 1, g] @ q[i, a]) * m["scale"], W["sink"][a])
        out[:, a] = P[a] @ v[:, g]
    if weights_out is not None:
        weights_out.append(P)
    return (out.reshape(T, H * vdim) * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


def plain_mlstm_gates(h, W, cap: float):
    """(log input gate, log forget gate) [T, heads]."""
    return (cap * torch.tanh((h @ W["i"].T + W["i.b"]) / cap),
            plain_log_sigmoid(cap * torch.tanh((h @ W["f"].T + W["f.b"]) / cap)))


def plain_mlstm_memory(q, k, v, i, f):
    """q (scaled), k [T, heads, dim], v [T, heads, vdim], i, f [T, heads] -> o [T, heads, vdim], one token after another."""
    T, H, dim = q.shape
    S = torch.zeros((H, dim, v.shape[2]), dtype=q.dtype)
    n = torch.zeros((H, dim), dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    outs = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, let = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + let[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + let[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        outs.append(torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None])
    return torch.stack(outs)


def plain_mlstm(h, W, m: dict, eps: float):
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ W["q"].T).reshape(T, H, dim) * dim ** -0.5
    i, f = plain_mlstm_gates(h, W, m["gate_cap"])
    o = plain_mlstm_memory(q, (h @ W["k"].T).reshape(T, H, dim), (h @ W["v"].T).reshape(T, H, vdim), i, f)
    y = plain_rms(o, eps).reshape(T, H * vdim) * W["norm"]
    return (y * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


def plain_gla_decays(h, W, tau: float):
    """[T, heads * dim]: the factor of every row of the state."""
    return torch.exp(plain_log_sigmoid((h @ W["a1"].T) @ W["a2"].T + W["a2.b"]) / tau)


def plain_gla_memory(q, k, v, a):
    """q (scaled), k, a [T, heads, dim], v [T, heads, vdim] -> o [T, heads, vdim], one token after another."""
    T, H, dim = q.shape
    S = torch.zeros((H, dim, v.shape[2]), dtype=q.dtype)
    outs = []
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        outs.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(outs)


def plain_gla(h, W, m: dict, eps: float):
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ W["q"].T).reshape(T, H, dim) * dim ** -0.5
    o = plain_gla_memory(q, (h @ W["k"].T).reshape(T, H, dim), (h @ W["v"].T).reshape(T, H, vdim),
                         plain_gla_decays(h, W, m["tau"]).reshape(T, H, dim))
    y = (plain_rms(o, eps) * W["norm"]).reshape(T, H * vdim)
    return (y * plain_silu(h @ W["g"].T)) @ W["o"].T


# ---------------------------------------------------------------------------------------------- feed-forwards
def plain_dense_ff(h, W):
    return (plain_gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def plain_route(s, correction, top: int, count: int, keep: int):
    """Scores s [n] of one token -> the chosen experts' indices.  Groups and experts are compared by s + correction."""
    c = s + correction
    per = c.numel() // count
    order = sorted(range(count), key=lambda g: -float(c[g * per:(g + 1) * per].max()))
    among = [e for g in order[:keep] for e in range(g * per, (g + 1) * per)]
    return sorted(among, key=lambda e: -float(c[e]))[:top]


def plain_moe(h, W, mlp: dict):
    r = mlp["router"]
    E, ident = r["experts"], r.get("identity", 0)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(h @ W["router"].T, dim=-1)
    corr = W.get("correction", torch.zeros(E + ident, dtype=h.dtype))
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in plain_route(s[t], corr, r["top"], groups["count"], groups["keep"]):
            if e >= E:
                y[t] += s[t, e] * h[t]
            else:
                z = plain_silu(W[f"e{e}.gate"] @ h[t]) * (W[f"e{e}.up"] @ h[t])
                y[t] += s[t, e] * (W[f"e{e}.down"] @ z)
    return y


# ---------------------------------------------------------------------------------------------- the model
def _sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def plain_forward(cfg: dict, weights: dict, ids, return_layers: bool = False, attention_out=None):
    """Logits [T, vocab] of one sequence (and the stream after every layer).  ``attention_out``: a dict that receives the
    softmax weights of every attention layer by its index."""
    eps = cfg["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(ids, dtype=torch.long)]
    streams, kept = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m, W = layer["mixer"], _sub(weights, p + "mix.")
        if layer["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                kept[i] = plain_keys_values(x, W, m, eps)
            seen = []
            y = plain_attention(x, W, m, eps, kept[i if src is None else src], seen)
            if attention_out is not None:
                attention_out[i] = seen[0]
        elif layer["type"] == "mlstm":
            y = plain_mlstm(x, W, m, eps)
        elif layer["type"] == "gla":
            y = plain_gla(x, W, m, eps)
        else:
            raise ValueError(f"unknown layer type {layer['type']!r}")
        x = x + plain_rms(y, eps) * weights[p + "norm1"]
        if layer.get("mlp") is not None:
            W = _sub(weights, p + "mlp.")
            y = plain_dense_ff(x, W) if layer["mlp"]["kind"] == "dense" else plain_moe(x, W, layer["mlp"])
            x = x + plain_rms(y, eps) * weights[p + "norm2"]
        streams.append(x)
    logits = (plain_rms(x, eps) * weights["final.norm"]) @ weights["embed"].T
    return (logits, torch.stack(streams)) if return_layers else logits
