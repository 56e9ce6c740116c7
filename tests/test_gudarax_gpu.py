"""The Gudarax design on the GPU: each new kernel or kernel option alone against a plain statement of it, then the model in
every cutting (whole, token by token, pieces down to two tokens, unequal batches, reused slots, pages and states, long
decoding), in 32-bit and in bfloat16, on configurations that differ in every size, and generation through the entry point."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import cima_b200
from cima_b200.cache.kv import KVCache, KVRequest
from cima_b200.engine import StepEntry
from cima_b200.engine.batch import build_batch
from gudarax_cases import CONFIGS, attention, config, folder, gpu_model, plain_weights, row_errors
from gudarax_plain import plain_delta_rule, plain_forward, plain_gelu_tanh, plain_slopes, plain_visible
from reference_kernels import ReferenceKernels
from helpers import random_tokens, run_batched, run_in_pieces, run_tail_one_by_one, run_whole

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEV = "cuda:0"
TOL = {"float32": 2e-4, "bfloat16": 6e-2}
_kernels, _models, _plain = [], {}, {}
R = ReferenceKernels()


def K():
    if not _kernels:
        from cima_b200.kernels import Kernels
        _kernels.append(Kernels(verbose=False))
    return _kernels[0]


def entries_batch(counts, starts, slots=None, device=DEV):
    slots = slots or list(range(len(counts)))
    return build_batch([StepEntry(s, [0] * c, []) for s, c in zip(slots, counts)], starts, 1 << 30, device)


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).abs().max()) <= tol * max(1.0, float(want.abs().max()))


def tol_of(dtype):
    return 2e-5 if dtype == "float32" else 1.2e-2


# ------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_with_position_vectors(dtype):
    torch.manual_seed(0)
    V, H, P = 50, 72, 90
    table, pos = torch.randn(V, H).to(DT[dtype]), torch.randn(P, H).to(DT[dtype])
    ids, at = torch.randint(0, V, (33,), dtype=torch.int32), torch.randint(0, P, (33,), dtype=torch.int32)
    want = table[ids.long()].float() * 1.7 + pos[at.long()].float()
    x, ssq, xw, w = (torch.empty(33, H, device=DEV), torch.empty(33, 1, device=DEV), torch.empty(33, H, dtype=torch.bfloat16, device=DEV), torch.rand(H))
    K().embed(ids.to(DEV), table.to(DEV), x, 1.7, ssq, w.to(DEV), xw, positions=pos.to(DEV), row_pos=at.to(DEV))
    assert close(x, want, 1e-6) and close(ssq[:, 0], (want ** 2).sum(1), 1e-5) and close(xw, want * w, 8e-3)
    K().embed(ids.to(DEV), table.to(DEV), x, 1.7)
    assert close(x, table[ids.long()].float() * 1.7, 1e-6)
    K().embed(ids.to(DEV), table.to(DEV), x, 1.0, positions=pos.to(DEV), row_pos=(at + 1000).to(DEV))          # beyond the table: its last row
    assert close(x, table[ids.long()].float() + pos[-1].float(), 1e-6)


@pytest.mark.parametrize("wdt,dtype", [("float32", "float32"), ("bfloat16", "bfloat16"), ("float32", "bfloat16")])
@pytest.mark.parametrize("T,W,dim,layers,layer", [(1, 96, 12, 3, 1), (8, 224, 16, 2, 0), (3, 100, 5, 4, 3), (5, 1536, 130, 2, 1), (2, 33, 1, 1, 0), (8, 3584, 256, 1, 0)])
def test_token_input_of_few_rows(T, W, dim, layers, layer, wdt, dtype):
    torch.manual_seed(W)
    V = 40
    x, w, table = torch.randn(T, W), (torch.randn(dim, W) * W ** -0.5).to(DT[wdt]), torch.randn(V, layers * dim).to(DT[dtype])
    toks = torch.randint(0, V, (T,), dtype=torch.int32)
    toks[0] = V - 1
    want = plain_gelu_tanh(x.double() @ w.double().T) * table[toks.long(), layer * dim:(layer + 1) * dim].double()
    z = torch.empty(T, dim, dtype=DT[dtype], device=DEV)
    K().token_side_few(x.to(DEV), w.to(DEV), table.to(DEV), toks.to(DEV), layer * dim, z, 1)
    assert close(z, want, tol_of(dtype))
    if T > 1:                                                    # a row does not depend on its neighbours
        one = torch.empty(1, dim, dtype=DT[dtype], device=DEV)
        K().token_side_few(x[1:2].to(DEV), w.to(DEV), table.to(DEV), toks[1:2].to(DEV), layer * dim, one, 1)
        assert torch.equal(one[0], z[1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,dim,layers,layer,act", [(9, 12, 3, 1, 1), (300, 16, 2, 1, 1), (70, 5, 3, 2, 0), (1000, 64, 1, 0, 1), (3, 6, 2, 1, 3)])
def test_token_input_applied_behind_a_product(T, dim, layers, layer, act, dtype):
    torch.manual_seed(T)
    V = 30
    z, table, toks = torch.randn(T, dim).to(DT[dtype]), torch.randn(V, layers * dim).to(DT[dtype]), torch.randint(0, V, (T,), dtype=torch.int32)
    want = R.gate_act(z.double(), act) * table[toks.long(), layer * dim:(layer + 1) * dim].double()
    got = z.to(DEV)
    K().token_side_apply(got, table.to(DEV), toks.to(DEV), layer * dim, act)
    assert close(got, want, tol_of(dtype))


def _cache(hd, nkv=1, dtype=torch.float32, tokens=64 * 16, window=0):
    return KVCache([[KVRequest(nkv, hd, window, 2)]], tokens, 1 << 20, dtype, DEV, page_size=64, max_seqs=4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,nkv,hd,dim,vd,first_hd", [(4, 2, 32, 24, 16, 0), (6, 2, 48, 40, 16, 32), (3, 3, 48, 16, 40, 48), (5, 1, 16, 8, 8, 16), (4, 2, 64, 64, 64, 80),
                                                     (28, 4, 128, 128, 128, 128), (40, 8, 128, 128, 100, 112), (2, 1, 144, 130, 7, 16)])
def test_norm_over_whole_projections_mixed_values_and_append(nh, nkv, hd, dim, vd, first_hd, dtype):
    torch.manual_seed(hd + nh)
    dt = DT[dtype]
    counts, starts = [9, 1, 70], [0, 77, 60]
    T = sum(counts)
    qkv = torch.randn(T, nh + 2 * nkv, hd)
    qkv[:, :nh + nkv, dim:] = 0.0
    qkv[:, nh + nkv:, vd:] = 0.0
    qkv = qkv.reshape(T, -1).to(dt)
    pad = lambda n: torch.nn.functional.pad(torch.rand(n, dim) + 0.5, (0, hd - dim)).reshape(-1)
    wq, wk = pad(nh), pad(nkv)
    first = torch.randn(T, nkv * max(first_hd, 1) + 8).to(dt)
    lam = torch.tensor([0.35])
    for mix in ([False, True] if first_hd else [False]):
        cache = _cache(hd, nkv, dt)
        slots = cache.open(3)
        for s, n, st in zip(slots, counts, starts):
            cache.reserve(s, st + n)
        cache.flush()
        batch, kv = entries_batch(counts, starts, slots), cache.layer_kv(0)
        firsts = first.to(DEV)[:, 4:]
        got = qkv.to(DEV)
        K().row_norm_append(got, (wq.to(DEV), wk.to(DEV), dim, 1e-3), batch, kv, nh, nkv, hd, vd, (lam.to(DEV), firsts, first_hd) if mix else None)
        x = qkv.double().view(T, nh + 2 * nkv, hd)
        q, k, v = x[:, :nh].reshape(T, -1), x[:, nh:nh + nkv].reshape(T, -1), x[:, nh + nkv:].clone()
        q = q / torch.sqrt((q * q).sum(1, keepdim=True) / (nh * dim) + 1e-3) * wq.double()
        k = k / torch.sqrt((k * k).sum(1, keepdim=True) / (nkv * dim) + 1e-3) * wk.double()
        if mix:
            f = first[:, 4:4 + nkv * first_hd].double().view(T, nkv, first_hd)
            v[..., :vd] = 0.65 * v[..., :vd] + 0.35 * f[..., :vd]
        want = torch.cat([q, k, v.reshape(T, -1)], 1)
        assert close(got, want, tol_of(dtype))
        for r, i, pos in ((0, 0, 0), (8, 0, 8), (9, 1, 77), (10, 2, 60), (13, 2, 63), (14, 2, 64), (79, 2, 129)):
            page = int(kv.block_table[slots[i], pos // 64])
            assert torch.equal(kv.storage[page, 0, :, pos % 64].reshape(-1), got[r, nh * hd:(nh + nkv) * hd])
            assert torch.equal(kv.storage[page, 1, :, pos % 64].reshape(-1), got[r, (nh + nkv) * hd:])


def test_norm_and_append_into_a_ring_of_pages():
    """A prompt longer than the ring: the ring holds its newest positions, each at its own place."""
    cache = _cache(32, 1, torch.float32, window=70)
    (slot,) = cache.open(1)
    cache.reserve(slot, 400); cache.flush()
    kv, batch = cache.layer_kv(0), entries_batch([400], [0], [slot])
    assert kv.ring_pages == 3
    torch.manual_seed(0)
    qkv = torch.randn(400, 96, device=DEV)
    K().row_norm_append(qkv, (torch.ones(32, device=DEV), torch.ones(32, device=DEV), 32, 1e-5), batch, kv, 1, 1, 32, 32)
    for pos in range(400 - 70, 400):
        page = int(kv.block_table[slot, (pos // 64) % 3])
        assert torch.equal(kv.storage[page, 0, 0, pos % 64], qkv[pos, 32:64]) and torch.equal(kv.storage[page, 1, 0, pos % 64], qkv[pos, 64:])


@pytest.mark.parametrize("window", [0, 1, 63, 64, 65, 130, 300])
@pytest.mark.parametrize("dtype,hd,nh,nkv", [("float32", 48, 4, 2), ("bfloat16", 48, 4, 2), ("bfloat16", 64, 4, 1), ("bfloat16", 128, 6, 2),
                                             ("bfloat16", 144, 2, 1), ("bfloat16", 96, 20, 1)])
def test_distance_slopes_through_every_attention_kernel(dtype, hd, nh, nkv, window):
    """A bias by distance, alone and beside a sink: prompts over their own rows (the plain, the tiled and, from 256 rows on, the
    tcgen05 kernel), rows that go on over the pages (tiled and tcgen05), single rows with one and with several splits.  Single
    scores stand out, on both sides of the window's edge among them."""
    torch.manual_seed(hd + nh)
    dt = DT[dtype]
    tol = 3e-5 if dtype == "float32" else 2.5e-2
    total, scale = 420, 0.35
    slopes = torch.tensor(plain_slopes(nh))
    q, k, v = (torch.randn(total, n, hd).to(dt) for n in (nh, nkv, nkv))
    for i in (100, 239, 299, 419):                                  # the oldest key inside and the first one outside the window
        for back in (window - 1, window, 200):
            if 0 < back <= i:
                k[i - back] = (q[i, ::nh // nkv].float() * 2.0).to(dt)
    rep = nh // nkv
    kk, vv = k.double().repeat_interleave(rep, 1), v.double().repeat_interleave(rep, 1)
    s = torch.einsum("ihd,jhd->hij", q.double(), kk) * scale
    dist = torch.arange(total)[:, None] - torch.arange(total)[None, :]
    s = s - torch.tensor(plain_slopes(nh), dtype=torch.float64)[:, None, None] * dist.double()
    seen = torch.zeros(total, total, dtype=torch.bool)
    for i in range(total):
        seen[i, plain_visible(i, window)] = True
    s = s.masked_fill(~seen, -float("inf"))
    rows = torch.cat([t.reshape(total, -1) for t in (q, k, v)], dim=1).to(DEV)
    cache = _cache(hd, nkv, dt)
    (slot,) = cache.open(1)
    kv = cache.layer_kv(0)
    cache.reserve(slot, total); cache.flush()
    for p in range(total):
        page = int(kv.block_table[slot, p // 64])
        kv.storage[page, 0, :, p % 64], kv.storage[page, 1, :, p % 64] = k[p].to(DEV), v[p].to(DEV)
    cache.commit(slot, total)
    for sink in (0.0, 1.0):
        full = torch.softmax(torch.cat([s, torch.zeros(nh, total, 1, dtype=torch.float64)], 2), 2)[:, :, :-1] if sink else torch.softmax(s, 2)
        want = torch.einsum("hij,jhd->ihd", full, vv).reshape(total, nh * hd)

        def run(lo, hi, from_cache):
            out = torch.empty(hi - lo, nh * hd, dtype=dt, device=DEV)
            K().attention(rows[lo:hi], kv, entries_batch([hi - lo], [lo], [slot]), out, nh, nkv, hd, scale, window, from_cache, sink=sink,
                          slopes=slopes.to(DEV))
            return out

        for n in (420, 300, 70, 1):
            assert close(run(0, n, n == 1), want[:n], tol), ("own rows", n)
        for lo, hi in ((200, 240), (120, 420), (419, 420), (100, 101), (298, 300)):
            assert close(run(lo, hi, True), want[lo:hi], tol), ("going on", lo, hi)
        if dtype == "bfloat16" and hd <= 128:
            b = entries_batch([1], [419], [slot])
            for splits in (1, 2, 5):
                out = torch.empty(1, nh * hd, dtype=dt, device=DEV)
                K().attention_decode(rows[419:420], kv, b.seq_slot, b.seq_len, out, nh, nkv, hd, scale, window, n_splits=splits, sink=sink,
                                     slopes=slopes.to(DEV))
                assert close(out, want[419:420], tol), ("splits", splits)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,heads,N,Kd,ha,ho", [(1, 3, 20, 40, 40, 20), (8, 2, 64, 128, 128, 64), (5, 4, 8, 17, 20, 10), (70, 3, 20, 40, 40, 20), (300, 4, 64, 64, 80, 64),
                                                (33, 2, 7, 24, 24, 9), (9, 28, 128, 128, 128, 128)])
def test_head_products_with_a_gate(T, heads, N, Kd, ha, ho, dtype):
    torch.manual_seed(T + N)
    dt = DT[dtype]
    a, w, g = torch.randn(T, heads * ha).to(dt), (torch.randn(heads, N, Kd) * Kd ** -0.5).to(dt), (torch.randn(T, heads * N + 24) * 2).to(dt)
    out = torch.full((T, heads * ho), 7.0, dtype=dt, device=DEV)
    K().head_linear(a.to(DEV), w.to(DEV), out, a_head=ha, out_head=ho, gate=(g.to(DEV), 16))
    for h in range(heads):
        want = (a[:, h * ha:h * ha + Kd].double() @ w[h].double().T) * torch.sigmoid(g[:, 16 + h * N:16 + (h + 1) * N].double())
        assert close(out[:, h * ho:h * ho + N], want, tol_of(dtype))
        assert bool((out[:, h * ho + N:(h + 1) * ho] == 7.0).all())                # what lies between the heads is left alone


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 16, 24), (2, 1, 128, 64), (3, 3, 40, 8), (2, 2, 200, 33), (6, 2, 64, 65), (2, 1, 1, 5), (1, 1, 13, 16)])
def test_delta_rule_with_one_decay_a_head_in_every_cutting(heads, kv_heads, dim, vdim, dtype):
    """From the convolved rows and slices of the projection on, against the rule in float64; whole, in pieces and token by token
    from the carried state and beside another sequence: the same bits."""
    torch.manual_seed(dim)
    T, kd = 75, kv_heads * dim
    c = torch.randn(T, 2 * kd + heads * vdim)
    c[50, kd:2 * kd] = c[3, kd:2 * kd]                                               # a key that is written again
    c[60, :2 * kd] = 0.0                                                             # rows without a direction
    c = c.to(DT[dtype])
    p = (torch.randn(T, 2 * heads + 7) * 2).to(DT[dtype])                            # b | a among other columns
    p[20, 3 + heads:3 + 2 * heads], p[30, 3:3 + heads] = 60.0, 40.0                  # a token that forgets all, one that writes all
    A, d = torch.randn(heads) * 1.5 - 1.0, torch.randn(heads)
    x = c.double()
    unit = lambda t: t / torch.sqrt((t * t).sum(-1, keepdim=True) + 1e-6)
    z = p[:, 3 + heads:3 + 2 * heads].double() + d.double()
    g = torch.exp(-torch.exp(A.double()) * (torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))))
    want = plain_delta_rule(unit(x[:, :kd].view(T, kv_heads, dim)) * dim ** -0.5, unit(x[:, kd:2 * kd].view(T, kv_heads, dim)),
                            x[:, 2 * kd:].view(T, heads, vdim), torch.sigmoid(p[:, 3:3 + heads].double()), g).reshape(T, -1)
    cd, pd, Ad, dd = c.to(DEV), p.to(DEV), A.to(DEV), d.to(DEV)

    def call(rows, st, batch):
        o = torch.empty(rows.stop - rows.start, heads * vdim, device=DEV)
        K().delta_rule(cd[rows], pd[rows, 3 + heads:3 + 2 * heads], pd[rows, 3:3 + heads], Ad, dd, st, batch, o, heads, kv_heads, dim, vdim)
        return o

    def run(counts):
        st, out, r = torch.zeros(4, heads, dim, vdim, device=DEV), [], 0
        for n in counts:
            out.append(call(slice(r, r + n), st, entries_batch([n], [r], [2])))
            r += n
        assert float(st[[0, 1, 3]].abs().max()) == 0.0
        return torch.cat(out), st

    out, st = run([T])
    assert close(out, want, 5e-6)
    bits = torch.equal if dtype == "float32" else lambda x, y: close(x, y, 5e-6)      # (long bfloat16 steps take 16 tokens at a time)
    for counts in ([2, 5, 33, 35], [1] * T, [16, 1, 58]):
        o2, s2 = run(counts)
        assert bits(o2, out) and bits(s2, st)
    if dtype == "bfloat16":
        (o1, s1), (o2, s2) = run([1] * T), run([31, 13, 31])
        assert torch.equal(o1, o2) and torch.equal(s1, s2)
    cd, pd = torch.cat([cd[:40], cd]), torch.cat([pd[:40], pd])
    st2 = torch.zeros(4, heads, dim, vdim, device=DEV)
    both = call(slice(0, 40 + T), st2, entries_batch([40, T], [0, 0], [3, 0]))
    assert torch.equal(both[40:], out) and bits(both[:40], out[:40]) and torch.equal(st2[0], st[2])


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 16, 24), (2, 1, 128, 64), (3, 3, 40, 8), (6, 2, 64, 72), (1, 1, 8, 16), (12, 12, 128, 128), (2, 2, 96, 200)])
def test_delta_rule_of_long_steps_sixteen_tokens_at_a_time(heads, kv_heads, dim, vdim):
    """Ragged sequences of whole and broken chunks from used states against the rule in float64 and the token kernel: decays from
    none to complete inside a chunk, keys written again, rows without a direction, alike keys one after another."""
    torch.manual_seed(dim + vdim)
    counts, slots = [33, 1, 160, 16, 47, 5], [3, 0, 5, 1, 7, 4]
    T, kd, H = sum(counts), kv_heads * dim, heads
    c = torch.randn(T, 2 * kd + H * vdim)
    c[45:50, kd:2 * kd] = c[44, kd:2 * kd]
    c[60, :2 * kd] = 0.0
    c[70, kd:2 * kd] *= 30.0
    c = c.bfloat16()
    p = torch.randn(T, 2 * H) * 2
    p[50:54, H:] = 80.0                                           # forget all, four tokens running
    p[90:110, H:] = -30.0                                         # forget nothing
    p[90:110, :H] = 30.0                                          # and write all
    p = p.bfloat16()
    A, d = torch.randn(H) * 1.5 - 1.0, torch.randn(H)
    st0 = torch.randn(8, H, dim, vdim)
    x = c.double()
    unit = lambda t: t / torch.sqrt((t * t).sum(-1, keepdim=True) + 1e-6)
    q, k, v = unit(x[:, :kd].view(T, kv_heads, dim)) * dim ** -0.5, unit(x[:, kd:2 * kd].view(T, kv_heads, dim)), x[:, 2 * kd:].view(T, H, vdim)
    z = p[:, H:].double() + d.double()
    g = torch.exp(-torch.exp(A.double()) * (torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))))
    beta = torch.sigmoid(p[:, :H].double())
    want, want_st, r = torch.empty(T, H, vdim, dtype=torch.float64), st0.double(), 0
    share = torch.arange(H) // (H // kv_heads)
    for n, s in zip(counts, slots):
        S = want_st[s]
        for t in range(r, r + n):
            kt, qt = k[t][share], q[t][share]
            S = g[t][:, None, None] * S
            u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, kt))
            S = S + kt[:, :, None] * u[:, None, :]
            want[t] = torch.einsum("hdv,hd->hv", S, qt)
        want_st[s] = S
        r += n
    cd, pd, Ad, dd = c.to(DEV), p.to(DEV), A.to(DEV), d.to(DEV)
    batch = entries_batch(counts, [9] * 6, slots)
    assert batch.max_rows >= K().DELTA_CHUNK_ROWS
    st, out = st0.to(DEV), torch.full((T, H * vdim), float("nan"), device=DEV)
    K().delta_rule(cd, pd[:, H:], pd[:, :H], Ad, dd, st, batch, out, H, kv_heads, dim, vdim)
    assert close(out, want.reshape(T, -1), 1e-5) and close(st, want_st, 1e-5)
    assert torch.equal(st[[2, 6]].cpu(), st0[[2, 6]])
    # token by token: the same but for rounding
    few, out2, r = st0.to(DEV), torch.empty(T, H * vdim, device=DEV), 0
    for n, s in zip(counts, slots):
        for lo in range(r, r + n, 20):
            hi = min(lo + 20, r + n)
            o = torch.empty(hi - lo, H * vdim, device=DEV)
            K().delta_rule(cd[lo:hi], pd[lo:hi, H:], pd[lo:hi, :H], Ad, dd, few, entries_batch([hi - lo], [9], [s]), o, H, kv_heads, dim, vdim)
            out2[lo:hi] = o
        r += n
    assert close(out2, out, 1e-5) and close(few, st, 1e-5)
    # beside others or alone: the same bits
    alone = st0.to(DEV)
    o = torch.empty(160, H * vdim, device=DEV)
    K().delta_rule(cd[34:194], pd[34:194, H:], pd[34:194, :H], Ad, dd, alone, entries_batch([160], [9], [5]), o, H, kv_heads, dim, vdim)
    assert torch.equal(o, out[34:194]) and torch.equal(alone[5], st[5])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,wide,taps", [(160, 200, 3), (96, 104, 4), (40, 43, 2), (64, 64, 1), (256, 320, 6)])
def test_short_convolution_on_column_slices(C, wide, taps, dtype):
    torch.manual_seed(C)
    p, w = torch.randn(120, wide).to(DT[dtype]), torch.randn(taps, C)
    want = torch.zeros(120, C, dtype=torch.float64)
    for j in range(taps):
        back = taps - 1 - j
        want[back:] += w[j].double() * p[:120 - back, :C].double()
    want = want * torch.sigmoid(want)
    pd = p.to(DEV)
    for rows_each in ([120], [1] * 120, [2, 50, 1, 67]):
        for per in (0, 8):
            st, out, r = torch.zeros(3, max(taps - 1, 1), C, dtype=DT[dtype], device=DEV), torch.empty(120, C, dtype=DT[dtype], device=DEV), 0
            for c in rows_each:
                o = torch.empty(c, C, dtype=DT[dtype], device=DEV)
                K().short_conv(pd[r:r + c, :C], w.to(DEV), st if taps > 1 else None, entries_batch([c], [r], [1]), o, per, add_input=False, act=0)
                out[r:r + c] = o
                r += c
            assert close(out, want, tol_of(dtype)), (rows_each[:3], per)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("gated,weigh_input,act", [(False, True, 5), (False, False, 5), (True, True, 0), (False, True, 1)])
@pytest.mark.parametrize("T,E,top,ff,H", [(4, 6, 2, 32, 96), (40, 5, 3, 24, 64), (100, 6, 2, 40, 72), (600, 8, 3, 64, 256), (3, 1, 1, 16, 30), (70, 4, 4, 9, 40),
                                          (1100, 3, 1, 96, 128)])
def test_ungated_experts_and_weights_on_inputs_on_every_road(T, E, top, ff, H, gated, weigh_input, act, dtype):
    torch.manual_seed(T)
    dt = DT[dtype]
    h = torch.randn(T, H).to(dt)
    gu, dn = (torch.randn(E, (2 if gated else 1) * ff, H) * H ** -0.5).to(dt), (torch.randn(E, H, ff) * ff ** -0.5).to(dt)
    idx = torch.stack([torch.randperm(E)[:top] for _ in range(T)]).to(torch.int32)
    wgt = torch.rand(T, top) * 0.9 + 0.1
    x = torch.zeros(T, H, dtype=torch.float64)
    for t in range(T):
        for j in range(top):
            e, w = int(idx[t, j]), float(wgt[t, j])
            z = gu[e].double() @ (h[t].double() * (w if weigh_input else 1.0))
            z = R.gated(z[:ff], z[ff:], act) if gated else R.ungated(z, act)
            x[t] += (1.0 if weigh_input else w) * (dn[e].double() @ z)
    for assign in (True, False):
        got = torch.full((T, H), 0.5, device=DEV)
        K().moe_experts(h.to(DEV), gu.to(DEV), dn.to(DEV), idx.to(DEV), wgt.to(DEV), got, act, assign=assign, gated=gated, weigh_input=weigh_input)
        assert close(got, x if assign else x + 0.5, 3e-5 if dtype == "float32" else 2.5e-2)
    assert K().device_errors() == 0


# ------------------------------------------------------------------------------------------- the model
def model_of(name, dtype, max_tokens=2048):
    """32-bit on the weights that make attention sharp; bfloat16 on the milder configuration of the same weights."""
    if (name, dtype) not in _models:
        _models[(name, dtype)] = gpu_model(name, dtype, max_tokens=max_tokens, sharp=dtype == "float32")
    return _models[(name, dtype)]


def plain_logits(name, toks, dtype="float32"):
    key = (name, tuple(toks), dtype == "float32")
    if key not in _plain:
        cfg, W = plain_weights(name, sharp=dtype == "float32")
        _plain[key] = plain_forward(cfg, W, toks)
    return _plain[key]


def agrees(got, want, dtype, what=""):
    e = row_errors(got, want)
    if dtype == "float32":
        assert e.max() < TOL[dtype], (what, float(e.max()))
    else:
        # a head of the delta rule is divided by its own size: where its read-out nearly cancels (q almost orthogonal to all that
        # is stored) bfloat16's rounding decides its direction; such rows are rare and the 32-bit runs compare every row sharply
        over = int((e >= 3 * TOL[dtype]).sum())
        assert e.median() < TOL[dtype] / 2 and over <= max(1, len(e) // 20) and e.max() < 1.0, (what, float(e.median()), float(e.max()), over)


LENGTHS = {"A": 150, "B": 131, "C": 330}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_and_token_by_token(name, dtype):
    cfg = CONFIGS[name]
    toks = random_tokens(cfg["vocab"], LENGTHS[name], seed=3)
    m = model_of(name, dtype)
    want = plain_logits(name, toks, dtype)
    agrees(run_whole(m, toks), want, dtype, "whole")
    agrees(run_tail_one_by_one(m, toks, 110), want, dtype, "tail")           # across pages' borders and the windows' edges
    agrees(run_tail_one_by_one(m, toks[:12], 12), want[:12], dtype, "first tokens")
    agrees(run_whole(m, toks[:1]), want[:1], dtype, "one token")
    m.cache.check()
    assert m.cache.slots.held == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_down_to_two_tokens(name, dtype):
    cfg = CONFIGS[name]
    a, b_ = random_tokens(cfg["vocab"], LENGTHS[name], seed=5), random_tokens(cfg["vocab"], 90, seed=6)
    m = model_of(name, dtype)
    got = run_in_pieces(m, [a, b_], [[2, 4, 7, 64, 66, 128, 129], [63, 65, 67]])
    agrees(got[0], plain_logits(name, a, dtype), dtype)
    agrees(got[1], plain_logits(name, b_, dtype), dtype)
    if dtype == "float32":                                                    # the cutting changes nothing but rounding
        assert row_errors(got[0], run_whole(m, a)).max() < 3e-5
    assert m.cache.slots.held == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_unequal_batches_on_reused_slots_pages_and_states(name, dtype):
    """Three rounds on a cache of three slots and few pages: later sequences get the slots, the pages and the states of earlier
    ones; shorter requests end earlier."""
    cfg = CONFIGS[name]
    m = gpu_model(name, dtype, max_tokens=64 * 6, max_seqs=3, sharp=dtype == "float32")
    for rnd in range(3):
        lens = [[5, 1, 130], [66, 3, 64], [1, 1, 63]][rnd]
        seqs = [random_tokens(cfg["vocab"], n + (2 if i == 1 else 9), seed=10 * rnd + i) for i, n in enumerate(lens)]
        got = run_batched(m, seqs, lens)
        for q, g_ in zip(seqs, got):
            agrees(g_, plain_logits(name, q, dtype), dtype, (rnd, len(q)))
        m.cache.check()
        assert m.cache.slots.held == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_of_more_rows_than_the_few_rows_kernels_take(dtype):
    cfg = CONFIGS["A"]
    m = gpu_model("A", dtype, max_tokens=64 * 24, max_seqs=12, sharp=dtype == "float32")
    seqs = [random_tokens(cfg["vocab"], 8 + 3 * i, seed=50 + i) for i in range(12)]
    got = run_batched(m, seqs, [max(1, len(q) - 8) for q in seqs])
    for q, g_ in zip(seqs, got):
        agrees(g_, plain_logits("A", q, dtype), dtype, len(q))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding(name, dtype):
    cfg = CONFIGS[name]
    toks = random_tokens(cfg["vocab"], 300, seed=9)
    agrees(run_tail_one_by_one(model_of(name, dtype), toks, 297), plain_logits(name, toks, dtype), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batch_composition_and_slot_do_not_change_a_row(dtype):
    cfg = CONFIGS["C"]
    m = model_of("C", dtype)
    a, others = random_tokens(cfg["vocab"], 140, seed=1), [random_tokens(cfg["vocab"], n, seed=n) for n in (300, 7)]
    alone = run_batched(m, [a], [130])[0]
    among = run_batched(m, [others[0], a, others[1]], [290, 130, 3])[1]
    e = row_errors(among, alone)
    if dtype == "float32":
        assert e.max() < 2e-5, float(e.max())
    else:
        assert e.median() < 2e-2 and e.max() < 0.1, (float(e.median()), float(e.max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_at_a_windows_edge(dtype, tmp_path):
    """One attention layer, two tokens whose key and query match: the later one's logits follow the earlier one's value while it
    lies inside the window (window - 1 back) and do not one position further, in prompts and in decoding, at page borders too."""
    from gudarax_cases import write_folder
    from gudarax_plain import read_folder
    from cima_b200.engine import load_model
    window = 70
    cfg = config(64, 64, 400, 1e-5, 1.0, 4, [attention(2, 1, 32, 32, 0.5, window, False, None)])
    d = write_folder(str(tmp_path), cfg, 5)
    from safetensors.torch import load_file, save_file
    path = os.path.join(d, "model.safetensors")
    t = load_file(path)
    gen = torch.Generator().manual_seed(0)
    rand = lambda *shape: torch.randn(*shape, generator=gen)
    E = rand(64, 64)
    E[:, 62:] = 0.0
    E[1], E[2] = 0.0, 0.0
    E[1, 62], E[2, 63] = 8.0, 8.0                                  # the query's token and the key's token: a column of their own each
    t["embed"], t["pos"] = E.to(torch.bfloat16), torch.zeros_like(t["pos"])
    u = rand(32)
    Wq, Wk = rand(64, 64), rand(32, 64)
    Wq[:, 62], Wk[:, 63] = torch.cat([u, u]), u                    # both heads of the one look for what the other has
    t["l0.mix.q"], t["l0.mix.k"] = Wq.to(torch.bfloat16), Wk.to(torch.bfloat16)
    for n in ("l0.mix.q.b", "l0.mix.k.b"):
        t[n] = torch.zeros_like(t[n])
    save_file({n: x.contiguous() for n, x in t.items()}, path)
    c, Wp = read_folder(d)
    m = load_model(d, dtype=dtype, max_tokens=1024, device=DEV, verbose=False)
    tol = 1e-4 if dtype == "float32" else 4e-2
    rng = np.random.default_rng(2)
    for at in (75, 128, 133, 200, 255):                            # where the query stands
        for back in (window - 1, window, 64, 1):
            toks = rng.integers(3, 64, size=at + 1).tolist()
            toks[at], toks[at - back] = 1, 2
            maps = {}
            want = plain_forward(c, Wp, toks, attention_out=maps)
            carried = float(maps[0][1, at, at - back])              # the head whose slope is small
            assert (carried > 0.5) if back < window else (carried == 0.0), (at, back, carried)
            for how, got in (("prompt", run_whole(m, toks)), ("decoded", run_tail_one_by_one(m, toks, 3)), ("piece", run_in_pieces(m, [toks], [[at - 40]])[0])):
                assert row_errors(got[at:], want[at:]).max() < tol, (how, at, back)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(dtype):
    name = "B"
    cfg, W = plain_weights(name, sharp=dtype == "float32")
    lm = cima_b200.load(folder(name, sharp=dtype == "float32"), dtype=dtype, max_tokens=1024, verbose=False)
    prompts = [random_tokens(cfg["vocab"], n, seed=40 + n) for n in (7, 1, 70, 64)]
    got = lm.generate(prompts, temperature=0, repeat_penalty=1.0, max_tokens=12)
    for p, r in zip(prompts, got):
        assert r.finish_reason == "length" and len(r.tokens) == 12
        seq, off = list(p), 0
        for t in r.tokens:
            lg = plain_forward(cfg, W, seq)[-1]
            spread = float((lg - lg.mean()).pow(2).mean().sqrt())
            off += int(lg[t] < lg.max() - (1e-4 if dtype == "float32" else 0.2 * spread))
            seq.append(t)
        assert off == 0
    assert lm.model.cache.slots.held == 0
    again = lm.generate(prompts[:2], temperature=0, repeat_penalty=1.0, max_tokens=12)     # on used slots, pages and states
    if dtype == "float32":
        assert [r.tokens for r in again] == [r.tokens for r in got[:2]]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_recorded_steps_give_what_single_steps_give(dtype):
    """Decoding from the recorded graph, prompts from recorded prompt steps (padded, the third time replayed), against the same
    tokens through the step function; past a window's edge and a page's border."""
    cfg = CONFIGS["A"]
    lm = cima_b200.load(folder("A", sharp=False), dtype=dtype, max_tokens=2048, verbose=False)
    assert lm.model.graph_safe and lm.stepper.use_graphs
    for rnd in range(3):
        prompt = random_tokens(cfg["vocab"], 25 + rnd, seed=70 + rnd)
        (r,) = lm.generate([prompt], temperature=0, repeat_penalty=1.0, max_tokens=60)
        seq = prompt + r.tokens
        lg = run_tail_one_by_one(lm.model, seq, len(r.tokens))
        for i, t in enumerate(r.tokens):
            row = lg[len(prompt) - 1 + i]
            spread = float((row - row.mean()).pow(2).mean().sqrt())
            assert row[t] >= row.max() - (1e-4 if dtype == "float32" else 0.1) * spread, (rnd, i)


def test_model_from_a_configuration_in_memory_and_its_tensors_by_name():
    lm = cima_b200.load(config=CONFIGS["A"], seed=4, dtype="float32", max_tokens=256, verbose=False)
    sd = {k: v.detach().cpu().double() for k, v in lm.model.state_dict().items()}
    toks = random_tokens(CONFIGS["A"]["vocab"], 20, seed=1)
    assert row_errors(run_whole(lm.model, toks), plain_forward(CONFIGS["A"], sd, toks)).max() < TOL["float32"]


def test_trace_replay_of_this_design(tmp_path):
    name = "A"
    V = CONFIGS[name]["vocab"]
    reqs = {"a": random_tokens(V, 70, seed=1), "b": random_tokens(V, 9, seed=2)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": reqs["a"][:66], "want": [0, 65]},
                                     {"id": "b", "tokens": reqs["b"][:5], "want": [4]}], "end": []}]
    for j in range(4):
        steps.append({"step": j + 1, "entries": [{"id": "a", "tokens": [reqs["a"][66 + j]], "want": [0]},
                                                 {"id": "b", "tokens": [reqs["b"][5 + j]], "want": [0]}],
                      "end": ["a", "b"] if j == 3 else []})
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder(name), "--dtype", "float32",
                        "--out", str(tmp_path), "--max-tokens", "256"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    wa, wb = plain_logits(name, reqs["a"]), plain_logits(name, reqs["b"])
    got = torch.from_numpy(np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(-1, V).copy())
    assert row_errors(got, torch.stack([wa[0], wa[65], wb[4]])).max() < TOL["float32"]
    got = torch.from_numpy(np.fromfile(tmp_path / "4.f32", dtype="<f4").reshape(-1, V).copy())
    assert row_errors(got, torch.stack([wa[69], wb[8]])).max() < TOL["float32"]
