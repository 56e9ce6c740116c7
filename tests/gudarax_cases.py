"""Small Gudarax configurations, their weights and helpers shared by the tests of that design.

The weights are drawn by ``cima_b200.write_random_model`` and then scaled by tensor name, so that softmax maps are sharp
(single keys carry rows, near or far), decays range from fast to slow, the token inputs and the position vectors are of the
stream's size, and experts differ."""
from __future__ import annotations

import os
import tempfile

import torch

import cima_b200
from cima_b200.engine import load_model


def latent(heads, dim, vdim, kv_rank, q_rank, scale, mlp):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, scale, window, v_mix, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(vocab, width, positions, eps, scale, side, layers):
    return {"architecture": "Gudarax", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "token_side": {"dim": side}, "layers": layers}


# every mixer and feed-forward; windows below and above a page; mixing layers of different key sizes (their heads are padded
# differently in the cache), one attention between them and one behind them that does not mix; a layer without feed-forward
G_A = config(300, 96, 640, 1e-6, 2.0, 12, [
    latent(3, 24, 20, 40, 28, 0.6, moe(5, 2, 32)),
    attention(4, 2, 24, 16, 0.7, 40, True, dense(72)),
    delta(4, 2, 16, 24, 3, None),
    attention(6, 2, 40, 16, 0.5, 100, True, moe(6, 1, 24)),
    attention(2, 1, 24, 24, 0.6, 0, False, moe(3, 3, 16))])
# a width that is no multiple of 8; one tap; ranks and a side size that are odd; one expert; a window of one position and one
# just above a page; key heads of their own for every head; value sizes above and below the key size
G_B = config(513, 100, 300, 1e-5, 1.0, 5, [
    delta(3, 1, 12, 20, 1, moe(1, 1, 16)),
    attention(3, 3, 16, 40, 1.1, 65, False, dense(33)),
    latent(2, 40, 8, 17, 9, 0.5, None),
    delta(2, 2, 40, 8, 5, dense(20)),
    attention(5, 1, 8, 8, 1.0, 1, True, None)])
# head sizes and ranks of 64 and 128 (the tensor-core attention's), windows that cross pages, a key size of 128 in the state
G_C = config(640, 224, 512, 1e-5, 0.5, 16, [
    attention(4, 2, 64, 64, 0.4, 130, True, dense(192)),
    latent(4, 64, 64, 128, 64, 0.35, moe(8, 4, 64)),
    delta(2, 1, 128, 64, 4, None),
    attention(2, 2, 128, 128, 0.3, 200, False, dense(96)),
    latent(2, 32, 64, 64, 48, 0.5, None),
    attention(2, 2, 64, 64, 0.4, 70, True, moe(8, 2, 40))])
CONFIGS = {"A": G_A, "B": G_B, "C": G_C}

# factor by the last part of a tensor's name (a drawn matrix has entries of about 0.02, the router of 0.1)
_BOOST = {"embed": 25.0, "pos": 40.0, "router": 1.5, "gate": 8.0, "up": 8.0, "g": 10.0, "b": 15.0, "a": 15.0, "conv": 2.0, "uq": 1.0, "uk": 1.0,
          "uv": 1.0, "proj": 1.0}
_DEFAULT_BOOST = 6.0


def _boost(name: str, t: torch.Tensor) -> torch.Tensor:
    last = name.rsplit(".", 1)[-1]
    if name == "side.embed":
        return t                                                # drawn with unit variance
    if last == "vmix":
        return (t.float() * 0.5 + 0.4).to(t.dtype)
    if last == "A_log":
        return (t.float() * 3.0 - 1.5).to(t.dtype)              # heads that forget at once beside heads that keep
    if t.dim() < 2:
        return (t.float() * 20.0).to(t.dtype) if last == "b" else t
    return (t.float() * _BOOST.get(last, _DEFAULT_BOOST)).to(t.dtype)


def _milder(cfg: dict) -> dict:
    import copy
    c = copy.deepcopy(cfg)
    for L in c["layers"]:
        if "scale" in L["mixer"]:
            L["mixer"]["scale"] /= 3.0
        if (L["mlp"] or {}).get("kind") == "moe":
            L["mlp"]["router"]["top"] = L["mlp"]["router"]["experts"]
    return c


_FOLDERS = {}


def write_folder(d: str, cfg: dict, seed: int = 0, sharp: bool = True) -> str:
    """A model folder of ``cfg``; ``sharp`` False divides the attentions' scales by 3 (queries and keys are normed, so the scale
    alone decides how sharp a map is) and lets every token use all experts: with sharp maps and close calls between experts
    the rounding of a row in bfloat16 decides which key carries it or which expert it takes, so bfloat16 runs are compared on
    the milder configuration."""
    from safetensors.torch import load_file, save_file
    cima_b200.write_random_model(d, cfg if sharp else _milder(cfg), seed=seed)
    path = os.path.join(d, "model.safetensors")
    save_file({n: _boost(n, t).contiguous() for n, t in load_file(path).items()}, path)
    return d


def folder(name: str, seed: int = 0, sharp: bool = True) -> str:
    key = (name, seed, sharp)
    if key not in _FOLDERS:
        _FOLDERS[key] = write_folder(tempfile.mkdtemp(prefix=f"cima_gudarax_{name}_"), CONFIGS[name], seed, sharp)
    return _FOLDERS[key]


def plain_weights(name: str, seed: int = 0, sharp: bool = True):
    """(config dict, tensors in float64) of a folder, read without the package."""
    from gudarax_plain import read_folder
    return read_folder(folder(name, seed, sharp))


def cpu_model(name, dtype="float32", max_tokens=1024, seed=0, sharp=True, **kw):
    from reference_kernels import ReferenceKernels
    return load_model(folder(name, seed, sharp), dtype=dtype, max_tokens=max_tokens, device="cpu", kernels=ReferenceKernels(),
                      verbose=False, **kw)


def gpu_model(name, dtype="float32", max_tokens=1024, seed=0, sharp=True, **kw):
    return load_model(folder(name, seed, sharp), dtype=dtype, max_tokens=max_tokens, device="cuda:0", verbose=False, **kw)


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Per row: root mean square of the difference (its mean taken off) over that of the wanted row."""
    d = got.double() - want.double()
    d = d - d.mean(dim=1, keepdim=True)
    w = want.double() - want.double().mean(dim=1, keepdim=True)
    return d.pow(2).mean(dim=1).sqrt() / w.pow(2).mean(dim=1).sqrt().clamp_min(1e-30)

