"""Small Pelatar configurations, their weights and helpers shared by the tests of that design.

The weights are drawn by ``cima_b200.write_random_model`` and then scaled by tensor name, so that softmax maps are sharp
(single keys carry rows, near or far), sinks take a share that differs from head to head, decays and forget gates range from
fast to slow, the memories' denominators stand on either side of their lower bound, and the router's choice hangs on its
correction."""
from __future__ import annotations

import os
import tempfile

import torch

import cima_b200
from cima_b200.engine import load_model


def attention(heads, kv_heads, dim, vdim, scale, temp, mlp, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def gla(heads, dim, vdim, tau, rank, mlp):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, groups=None):
    r = {"experts": experts, "identity": identity, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def config(vocab, width, eps, layers):
    return {"architecture": "Pelatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# every mixer and feed-forward; grouped key heads, two readers of one layer's keys and values (one behind a memory layer);
# value sizes above and below the key size; a temperature that steps within the first page; a layer without feed-forward
P_A = config(300, 96, 1e-6, [
    gla(3, 24, 40, 4.0, 8, dense(72)),
    attention(4, 2, 24, 16, 0.9, (0.4, 16), moe(5, 3, 2, 32, (4, 2))),
    attention(4, 2, 24, 16, 0.8, (0.2, 50), dense(40), kv_from=1),
    mlstm(2, 16, 24, 10.0, None),
    attention(4, 2, 24, 16, 1.0, None, moe(6, 2, 3, 24, (2, 1)), kv_from=1)])
# a width that is no multiple of 8; one key head for all; one head; one expert beside one identity expert; every expert
# chosen; a temperature that steps at every position; a decay's exponent of 1 and a rank of 3; a small cap
P_B = config(513, 100, 1e-5, [
    mlstm(3, 8, 20, 5.0, moe(1, 1, 1, 16)),
    attention(3, 1, 16, 40, 1.1, None, None),
    gla(1, 40, 8, 1.0, 3, moe(5, 2, 7, 8)),
    attention(2, 2, 40, 40, 0.5, (0.1, 1), dense(33)),
    gla(5, 12, 12, 16.0, 5, None)])
# heads of 64 and 128 values (the tensor-core attention's sizes) and a reader of their keys; key sizes of 128 and above in
# the memories; groups of one expert; only identity experts in the last group; as many identity experts as others
P_C = config(640, 224, 1e-5, [
    attention(4, 1, 64, 64, 0.5, (0.3, 100), moe(8, 8, 4, 64, (16, 9))),
    mlstm(2, 128, 64, 15.0, dense(192)),
    gla(2, 64, 128, 16.0, 16, moe(6, 2, 2, 40, (4, 3))),
    attention(2, 2, 128, 128, 0.35, (0.5, 64), None),
    attention(2, 2, 128, 128, 0.3, None, dense(96), kv_from=3),
    mlstm(1, 160, 36, 8.0, None)])
CONFIGS = {"A": P_A, "B": P_B, "C": P_C}

# factor by the last part of a tensor's name (a drawn matrix has entries of about 0.02, the low-rank second factor and the
# router of 0.1)
_BOOST = {"embed": 40.0, "a1": 10.0, "a2": 3.0, "router": 1.5, "gate": 15.0, "up": 15.0, "g": 10.0, "i": 12.0, "f": 12.0}
_DEFAULT_BOOST = 6.0


def _boost(name: str, t: torch.Tensor, sharp: bool = True) -> torch.Tensor:
    last = name.rsplit(".", 1)[-1]
    if last == "correction":
        # sharp: of the size of the softmax scores' differences, so that the choice hangs on both; else above them, so that no
        # rounding turns it
        return (t.float() * (8.0 if sharp else 100.0)).to(t.dtype)
    if name.endswith("f.b"):
        return (t.float() + 2.0).to(t.dtype)                # forget gates that keep
    if last == "sink":
        return (t.float() * (2.0 if sharp else 1.0)).to(t.dtype)
    if t.dim() < 2:
        return t
    return (t.float() * _BOOST.get(last, _DEFAULT_BOOST)).to(t.dtype)


def _milder(cfg: dict) -> dict:
    import copy
    c = copy.deepcopy(cfg)
    for L in c["layers"]:
        if L["type"] == "attention":
            L["mixer"]["scale"] /= 3.0
    return c


_FOLDERS = {}


def write_folder(d: str, cfg: dict, seed: int = 0, sharp: bool = True) -> str:
    """A model folder of ``cfg``; ``sharp`` False divides the attention's scales by 3 (q and k are unit vectors up to a factor,
    so the scale alone decides how sharp a map is): with sharp maps the rounding of a query in bfloat16 decides which key
    carries a row, so bfloat16 runs are compared on the milder configuration."""
    from safetensors.torch import load_file, save_file
    cima_b200.write_random_model(d, cfg if sharp else _milder(cfg), seed=seed)
    path = os.path.join(d, "model.safetensors")
    save_file({n: _boost(n, t, sharp).contiguous() for n, t in load_file(path).items()}, path)
    return d


def folder(name: str, seed: int = 0, sharp: bool = True) -> str:
    key = (name, seed, sharp)
    if key not in _FOLDERS:
        _FOLDERS[key] = write_folder(tempfile.mkdtemp(prefix=f"cima_pelatar_{name}_"), CONFIGS[name], seed, sharp)
    return _FOLDERS[key]


def plain_weights(name: str, seed: int = 0, sharp: bool = True):
    """(config dict, tensors in float64) of a folder, read without the package."""
    from pelatar_plain import read_folder
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
