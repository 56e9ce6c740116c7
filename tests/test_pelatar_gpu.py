"""The Pelatar design on the GPU: each new kernel or kernel option alone against a plain statement of it, then the model in
every cutting (whole, token by token, pieces down to two tokens, unequal batches, reused slots, pages and states, long
decoding, prompts long enough to be cut into segments), in 32-bit and in bfloat16, on configurations that differ in every
size, and generation through the entry point."""
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
from pelatar_cases import CONFIGS, folder, gpu_model, plain_weights, row_errors
from pelatar_plain import plain_forward, plain_query_temperature
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
@pytest.mark.parametrize("T,W", [(1, 40), (7, 96), (300, 512), (5, 1536), (3, 101), (9, 2048), (2, 3584), (2, 8192), (2, 8200), (4, 1)])
def test_norm_on_a_branch_with_the_next_readers_rows(T, W, dtype):
    torch.manual_seed(T + W)
    x, y, w, w2 = torch.randn(T, W) * 3, torch.randn(T, W) * 0.2, torch.rand(W) + 0.5, torch.rand(W) + 0.5
    for follow in (None, (w2, 1e-4)):
        for rows in (True, False):
            if follow is not None and not rows:
                continue
            want_x, want_h = x.clone(), torch.empty(T, W)
            R.branch_norm(want_x, y, w, 1e-3, want_h, follow)
            got_x, got_h = x.to(DEV), torch.empty(T, W, dtype=DT[dtype], device=DEV)
            K().branch_norm(got_x, y.to(DEV), w.to(DEV), 1e-3, got_h if rows else None, None if follow is None else (w2.to(DEV), 1e-4))
            assert close(got_x, want_x, 2e-6)
            if rows:
                assert close(got_h, want_h, tol_of(dtype))


@pytest.mark.parametrize("gate_dtype,out_dtype", [("float32", "float32"), ("bfloat16", "bfloat16"), ("float32", "bfloat16")])
@pytest.mark.parametrize("T,G,n", [(3, 4, 24), (70, 2, 128), (5, 3, 200), (2, 1, 300), (4, 2, 700), (1, 6, 33)])
def test_heads_normed_and_gated(T, G, n, gate_dtype, out_dtype):
    torch.manual_seed(n)
    o = torch.randn(T, G * n)
    wide = (torch.randn(T, G * n + 11) * 2).to(DT[gate_dtype])
    den, low = torch.randn(T, G) * 2, torch.rand(T, G) + 0.05
    for w in (torch.rand(n) + 0.5, torch.rand(G * n) + 0.5):
        for silu in (False, True):
            for div in (None, (den, low, 1e-6)):
                want = torch.empty(T, G * n)
                R.group_rmsnorm_gate(o, w, wide[:, 3:3 + G * n], want, G, 0.05, silu=silu, divisor=div)
                got = torch.empty(T, G * n, dtype=DT[out_dtype], device=DEV)
                wd = wide.to(DEV)
                K().group_rmsnorm_gate(o.to(DEV), w.to(DEV), wd[:, 3:3 + G * n], got, G, 0.05, silu=silu,
                                       divisor=None if div is None else (den.to(DEV), low.to(DEV), 1e-6))
                assert close(got, want, tol_of(out_dtype))


@pytest.mark.parametrize("adt,wdt", [("float32", "float32"), ("float32", "bfloat16"), ("bfloat16", "bfloat16")])
@pytest.mark.parametrize("T,C,rank,tau", [(1, 40, 3, 1.0), (8, 384, 16, 16.0), (300, 129, 5, 4.0), (17, 200, 64, 16.0), (100, 130, 8, 16.0), (70, 40, 17, 2.0)])
def test_channel_decays(T, C, rank, tau, adt, wdt):
    torch.manual_seed(C)
    a1 = (torch.randn(T, rank + 9) * 2).to(DT[adt])
    w2, b = torch.randn(C, rank).to(DT[wdt]), torch.randn(C) * 2
    b[0], b[1] = 90.0, -90.0                                    # both tails of the sigmoid
    want, got = torch.empty(T, C), torch.empty(T, C, device=DEV)
    R.channel_decay(a1[:, 4:4 + rank].double(), w2.double(), b.double(), tau, want)
    a1d = a1.to(DEV)
    K().channel_decay(a1d[:, 4:4 + rank], w2.to(DEV), b.to(DEV), tau, got)
    assert float((got.cpu() - want).abs().max()) < 2e-6


def _memory_inputs(T, heads, dim, vdim, dtype, seed):
    torch.manual_seed(seed)
    p = torch.randn(T, heads * (2 * dim + vdim) + 5)
    return p.to(DT[dtype])


def _memory_views(p, heads, dim, vdim):
    a, b = heads * dim, 2 * heads * dim
    return p[:, :a], p[:, a:b], p[:, b:b + heads * vdim]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 24, 40), (3, 64, 64), (1, 128, 100), (2, 200, 33), (4, 8, 8), (2, 160, 130)])
@pytest.mark.parametrize("scalar", [False, True])
def test_memories_in_every_cutting(scalar, heads, dim, vdim, dtype):
    """Whole, in pieces and token by token from the carried state, and beside another sequence; the whole run is also compared
    with a plain statement of the recurrence in float64."""
    T = 75
    p = _memory_inputs(T, heads, dim, vdim, dtype, dim)
    q, k, v = _memory_views(p, heads, dim, vdim)
    pd = p.to(DEV)
    qd, kd, vd = _memory_views(pd, heads, dim, vdim)
    if scalar:
        g = torch.stack([torch.rand(T, heads) * 0.5 + 0.5, torch.rand(T, heads)], dim=-1)
    else:
        g = torch.rand(T, heads * dim) ** 0.2
    gd = g.to(DEV)
    scale = dim ** -0.5

    def run(counts, start_state=None):
        st = torch.zeros(4, heads, dim, vdim, device=DEV)
        ns = torch.zeros(4, heads, dim, device=DEV)
        out, den, r = torch.empty(T, heads * vdim, device=DEV), torch.empty(T, heads, device=DEV), 0
        for c in counts:
            b = entries_batch([c], [r], [2])
            o, d = torch.empty(c, heads * vdim, device=DEV), torch.empty(c, heads, device=DEV)
            K().memory(qd[r:r + c], kd[r:r + c], vd[r:r + c], gd[r:r + c].contiguous(), st, b, o, heads, dim, vdim, scale,
                       norm_state=ns if scalar else None, norm_out=d if scalar else None)
            out[r:r + c], den[r:r + c] = o, d
            r += c
        assert float(st[[0, 1, 3]].abs().max()) == 0.0 and float(ns[[0, 1, 3]].abs().max()) == 0.0
        return out, den, st, ns

    out, den, st, ns = run([T])
    S, n = torch.zeros(heads, dim, vdim, dtype=torch.float64), torch.zeros(heads, dim, dtype=torch.float64)
    qf, kf, vf = (t.double().reshape(T, heads, -1) for t in (q, k, v))
    want, wden = torch.empty(T, heads, vdim, dtype=torch.float64), torch.empty(T, heads, dtype=torch.float64)
    for t in range(T):
        gt = g[t].double()
        a = gt[:, 0, None].expand(heads, dim) if scalar else gt.view(heads, dim)
        kk = kf[t] * gt[:, 1, None] if scalar else kf[t]
        S = a[:, :, None] * S + kk[:, :, None] * vf[t][:, None, :]
        n = a * n + kk
        want[t], wden[t] = torch.einsum("hdv,hd->hv", S, qf[t]) * scale, (n * qf[t]).sum(-1) * scale
    assert close(out, want.reshape(T, -1), 3e-6) and close(st[2], S, 3e-6)
    if scalar:
        assert close(den, wden, 3e-6) and close(ns[2], n, 3e-6)
    for counts in ([2, 5, 33, 35], [1] * T, [16, 1, 58]):
        o2, d2, s2, n2 = run(counts)
        assert torch.equal(o2, out) and torch.equal(s2, st)                              # the same bits in every cutting
        if scalar:
            assert torch.equal(d2, den) and torch.equal(n2, ns)
    # beside another sequence, on other slots
    pb = torch.cat([p[:40], p]).to(DEV)
    qb, kb, vb = _memory_views(pb, heads, dim, vdim)
    gb = torch.cat([g[:40], g]).to(DEV)
    st2, ns2 = torch.zeros(4, heads, dim, vdim, device=DEV), torch.zeros(4, heads, dim, device=DEV)
    o, d = torch.empty(40 + T, heads * vdim, device=DEV), torch.empty(40 + T, heads, device=DEV)
    K().memory(qb, kb, vb, gb, st2, entries_batch([40, T], [0, 0], [3, 0]), o, heads, dim, vdim, scale,
               norm_state=ns2 if scalar else None, norm_out=d if scalar else None)
    assert torch.equal(o[40:], out) and torch.equal(st2[0], st[2])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 24, 40), (1, 128, 130), (2, 160, 33), (3, 64, 64)])
@pytest.mark.parametrize("scalar", [False, True])
def test_memories_cut_into_segments(scalar, heads, dim, vdim, dtype):
    """Steps long enough to be cut: sequences of several segments, of exactly two, of one token more, and a short one in the same
    step, from a used state; against the uncut kernel token after token."""
    seg = K().MEMORY_SEGMENT
    counts = [2 * seg, 3 * seg + 1, 5, 2 * seg - 1]
    T = sum(counts)
    p = _memory_inputs(T, heads, dim, vdim, dtype, dim + 1).to(DEV)
    q, k, v = _memory_views(p, heads, dim, vdim)
    torch.manual_seed(7)
    g = (torch.stack([torch.rand(T, heads) * 0.02 + 0.98, torch.rand(T, heads)], dim=-1) if scalar else torch.rand(T, heads * dim) ** 0.02).to(DEV)
    st0 = torch.randn(5, heads, dim, vdim, device=DEV)
    ns0 = torch.randn(5, heads, dim, device=DEV)
    slots = [3, 0, 4, 1]

    def run(cut):
        st, ns = st0.clone(), ns0.clone()
        out, den = torch.empty(T, heads * vdim, device=DEV), torch.empty(T, heads, device=DEV)
        if cut:
            b = entries_batch(counts, [0] * 4, slots)
            assert K().memory_segments(b) == 4
            K().memory(q, k, v, g, st, b, out, heads, dim, vdim, dim ** -0.5, norm_state=ns if scalar else None, norm_out=den if scalar else None)
            return out, den, st, ns
        r = 0
        for c, s in zip(counts, slots):
            for lo in range(0, c, seg):
                n = min(seg, c - lo)
                x = slice(r + lo, r + lo + n)
                o, d = torch.empty(n, heads * vdim, device=DEV), torch.empty(n, heads, device=DEV)
                K().memory(q[x], k[x], v[x], g[x].contiguous(), st, entries_batch([n], [lo], [s]), o, heads, dim, vdim, dim ** -0.5,
                           norm_state=ns if scalar else None, norm_out=d if scalar else None)
                out[x], den[x] = o, d
            r += c
        return out, den, st, ns

    (o1, d1, s1, n1), (o2, d2, s2, n2) = run(True), run(False)
    assert close(o1, o2, 1e-5) and close(s1, s2, 1e-5)
    assert torch.equal(s1[2], st0[2]) and torch.equal(n1[2], ns0[2])                       # a slot of no sequence is left alone
    if scalar:
        assert close(d1, d2, 1e-5) and close(n1, n2, 1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,heads,cap", [(1, 3, 5.0), (100, 2, 15.0), (33, 5, 8.0), (500, 3, 15.0), (448, 2, 6.0)])
def test_scalar_gates_in_every_cutting(T, heads, cap, dtype):
    torch.manual_seed(T)
    z = (torch.randn(T, 2 * heads + 3) * 6).to(DT[dtype])
    bi, bf = torch.randn(heads), torch.randn(heads) + 2
    want_ab, want_low, m = torch.empty(T, heads, 2), torch.empty(T, heads), torch.zeros(3, heads)
    R.scalar_gates(z.float(), bi, bf, cap, m, entries_batch([T], [0], [1], "cpu"), want_ab, want_low)
    zd = z.to(DEV)
    first = None
    for counts in ([T], [1] * T, [T - T // 3] + ([T // 3] if T // 3 else [])):
        md = torch.zeros(3, heads, device=DEV)
        ab, low, r = torch.empty(T, heads, 2, device=DEV), torch.empty(T, heads, device=DEV), 0
        for c in counts:
            a, l = torch.empty(c, heads, 2, device=DEV), torch.empty(c, heads, device=DEV)
            K().scalar_gates(zd[r:r + c], bi.to(DEV), bf.to(DEV), cap, md, entries_batch([c], [r], [1]), a, l)
            ab[r:r + c], low[r:r + c] = a, l
            r += c
        assert close(ab, want_ab, 2e-5) and close(low, want_low, 2e-5) and close(md[1], m[1], 2e-6)
        assert float(md[0].abs().max()) == 0.0
        if first is None:
            first = (ab, low, md)
        assert torch.equal(ab, first[0]) and torch.equal(low, first[1]) and torch.equal(md, first[2])


def _cache(hd, nkv=1, dtype=torch.float32, tokens=64 * 12):
    return KVCache([[KVRequest(nkv, hd, 0, 2)]], tokens, 1 << 20, dtype, DEV, page_size=64, max_seqs=4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,nkv,hd,norm_dim,rot", [(4, 2, 32, 24, 0), (3, 1, 40, 40, 0), (2, 2, 128, 128, 64), (6, 0, 48, 40, 0), (2, 1, 21, 17, 8),
                                                     (12, 2, 128, 128, 0), (20, 3, 64, 58, 0), (3, 1, 144, 140, 0), (9, 0, 64, 64, 0)])
def test_weightless_norm_temperature_and_append(nh, nkv, hd, norm_dim, rot, dtype):
    torch.manual_seed(hd)
    dt = DT[dtype]
    cache = _cache(hd, max(nkv, 1), dt)
    slots = cache.open(3)
    counts, starts = [9, 1, 70], [0, 77, 60]
    for s, n, st in zip(slots, counts, starts):
        cache.reserve(s, st + n)
    cache.flush()
    batch = entries_batch(counts, starts, slots)
    T, cols = sum(counts), (nh + 2 * nkv) * hd
    qkv = torch.randn(T, cols + 24).to(dt)                                       # columns behind the heads (a gate) stay as they are
    inv = torch.tensor([50.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float32)
    for temp in (None, (0.4, 16), (0.25, 1)):
        want, got = qkv.clone(), qkv.to(DEV)
        R.rope_append(want, inv, rot, *(getattr(batch, n).cpu() for n in ("row_pos", "row_seq", "seq_slot", "seq_len")), None, nh, nkv, hd,
                      qk_norm=(None, None, norm_dim, 1e-3), q_temp=temp)
        K().rope_append(got, inv.to(DEV), rot, batch.row_pos, batch.row_seq, batch.seq_slot, batch.seq_len, cache.layer_kv(0) if nkv else None,
                        nh, nkv, hd, qk_norm=(None, None, norm_dim, 1e-3), q_temp=temp)
        assert close(got, want, tol_of(dtype))
        assert torch.equal(got[:, cols:].cpu(), qkv[:, cols:])
    # the queries' factor written out, on rows of one sequence that goes on at position 60
    if rot == 0:
        q0 = qkv[10:, :norm_dim].double()
        plain = q0 / torch.sqrt((q0 * q0).mean(-1, keepdim=True) + 1e-3)
        factor = torch.tensor([plain_query_temperature(60 + t, 0.25, 1) for t in range(70)], dtype=torch.float64)
        assert close(got[10:, :norm_dim], plain * factor[:, None], tol_of(dtype))
    if nkv:
        kv = cache.layer_kv(0)
        for r, pos in ((9, 77), (10, 60), (79, 129)):
            page = int(kv.block_table[slots[1 if r == 9 else 2], pos // 64])
            assert close(kv.storage[page, 0, :, pos % 64].reshape(-1), want[r, nh * hd:(nh + nkv) * hd], tol_of(dtype))
            assert torch.equal(kv.storage[page, 1, :, pos % 64].reshape(-1).cpu(), qkv[r, (nh + nkv) * hd:cols])


@pytest.mark.parametrize("dtype,hd,nh,nkv", [("float32", 48, 4, 2), ("bfloat16", 48, 4, 2), ("bfloat16", 64, 4, 1), ("bfloat16", 128, 4, 2),
                                             ("bfloat16", 80, 3, 3), ("bfloat16", 144, 2, 1), ("float32", 40, 2, 1)])
def test_a_rows_own_gate_through_every_attention_kernel(dtype, hd, nh, nkv):
    """A gate value for every value of a row's result, read from the row's own buffer, beside a stored number a head in the
    softmax: prompts over their own rows (the plain, the tiled and, from 256 rows on, the tcgen05 kernel), rows that go on over
    the pages (tiled and tcgen05), single rows with one and with several splits, rows without keys of their own."""
    torch.manual_seed(hd + nh)
    dt = DT[dtype]
    tol = 3e-5 if dtype == "float32" else 2.5e-2
    sinks = torch.randn(nh) * 2.0
    total, scale = 420, 0.35
    q, k, v, g = (torch.randn(total, n, hd).to(dt) for n in (nh, nkv, nkv, nh))
    rep = nh // nkv
    kk, vv = k.double().repeat_interleave(rep, 1), v.double().repeat_interleave(rep, 1)
    s = torch.einsum("ihd,jhd->hij", q.double(), kk) * scale
    s = s.masked_fill(torch.ones(total, total).triu(1).bool(), -float("inf"))
    full = torch.softmax(torch.cat([s, sinks.double()[:, None, None].expand(nh, total, 1)], dim=2), dim=2)[:, :, :-1]
    want = (torch.einsum("hij,jhd->ihd", full, vv) * torch.sigmoid(g.double())).reshape(total, nh * hd)
    flat = lambda t: t.reshape(total, -1)
    rows = torch.cat([flat(q), flat(k), flat(v), flat(g)], dim=1).to(DEV)
    alone = torch.cat([flat(q), flat(g)], dim=1).to(DEV)
    col, col_alone = (nh + 2 * nkv) * hd, nh * hd
    cache = _cache(hd, nkv, dt)
    (slot,) = cache.open(1)
    kv = cache.layer_kv(0)
    cache.reserve(slot, total); cache.flush()
    for p in range(total):
        page = int(kv.block_table[slot, p // 64])
        kv.storage[page, 0, :, p % 64], kv.storage[page, 1, :, p % 64] = k[p].to(DEV), v[p].to(DEV)
    cache.commit(slot, total)

    def run(buf, gate_col, lo, hi, from_cache):
        out = torch.empty(hi - lo, nh * hd, dtype=dt, device=DEV)
        K().attention(buf[lo:hi], kv, entries_batch([hi - lo], [lo], [slot]), out, nh, nkv, hd, scale, 0, from_cache,
                      head_sink=sinks.to(DEV), gate_col=gate_col)
        return out

    for n in (300, 70, 1):
        assert close(run(rows, col, 0, n, n == 1), want[:n], tol), ("own rows", n)
        assert close(run(alone, col_alone, 0, n, True), want[:n], tol), ("another's keys", n)
    for lo, hi in ((200, 240), (120, 420), (419, 420), (100, 101)):
        assert close(run(rows, col, lo, hi, True), want[lo:hi], tol), ("going on", lo, hi)
        assert close(run(alone, col_alone, lo, hi, True), want[lo:hi], tol), ("going on, another's keys", lo, hi)
    if dtype == "bfloat16" and hd <= 128:
        b = entries_batch([1], [419], [slot])
        for splits in (1, 2, 5):
            out = torch.empty(1, nh * hd, dtype=dt, device=DEV)
            K().attention_decode(rows[419:420], kv, b.seq_slot, b.seq_len, out, nh, nkv, hd, scale, 0, n_splits=splits,
                                 head_sink=sinks.to(DEV), gate_col=col)
            assert close(out, want[419:420], tol), ("splits", splits)


@pytest.mark.parametrize("T,E,real,top,groups,keep", [(5, 8, 5, 2, 4, 2), (70, 16, 12, 3, 2, 1), (3, 2, 1, 1, 1, 1), (300, 24, 16, 6, 8, 3),
                                                      (9, 7, 5, 7, 1, 1), (20, 12, 8, 2, 12, 2), (64, 200, 150, 8, 10, 4)])
def test_routing_over_experts_and_identity_experts(T, E, real, top, groups, keep):
    torch.manual_seed(E)
    pad = -E % 8
    scores, corr = torch.randn(T, E + pad) * 2, torch.randn(E) * 0.2
    wi, ww = torch.empty(T, top, dtype=torch.int32), torch.empty(T, top)
    R.moe_route(scores.clone(), top, groups, keep, 1.0, wi, ww, experts=E, softmax=True, correction=corr, real=real, best_one=True, divide=False)
    for order in (False, True):
        gi, gw = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
        meta = K().moe_route(scores.to(DEV), top, groups, keep, 1.0, gi, gw, order=order and T <= 64, experts=E, softmax=True,
                             correction=corr.to(DEV), real=real, best_one=True, divide=False)
        pick = torch.zeros(T, E).scatter_(1, wi.long(), ww)
        assert close(torch.zeros(T, E).scatter_(1, gi.cpu().long(), gw.cpu()), pick, 1e-5)
        if meta is not None:                                                     # the pairs in the products are the experts' own
            assert int(meta[real]) == int((gi < real).sum())
            perm = meta[2 * (real + 1):][:int(meta[real])].cpu().long()
            assert torch.equal(perm.sort().values, torch.nonzero(gi.cpu().reshape(-1) < real)[:, 0])
    s = torch.softmax(scores[:, :E], dim=1)
    assert close(ww, torch.gather(s, 1, wi.long()), 1e-6)                       # the scores as they are


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,E,identity,top,ff,H", [(4, 6, 2, 2, 32, 96), (40, 5, 5, 3, 24, 64), (100, 6, 1, 2, 40, 72), (600, 8, 4, 3, 64, 256),
                                                   (3, 1, 1, 2, 16, 30), (7, 3, 9, 10, 8, 40)])
def test_experts_beside_identity_experts_on_every_road(T, E, identity, top, ff, H, dtype):
    torch.manual_seed(T)
    dt = DT[dtype]
    h = torch.randn(T, H).to(dt)
    gu, dn = (torch.randn(E, 2 * ff, H) * 0.3).to(dt), (torch.randn(E, H, ff) * 0.2).to(dt)
    idx = torch.stack([torch.randperm(E + identity)[:top] for _ in range(T)]).to(torch.int32)
    idx[0] = torch.arange(E + identity - top, E + identity)                       # a row of identity experts, as far as they go
    wgt = torch.rand(T, top)
    for assign in (True, False):
        want = torch.full((T, H), 0.5)
        R.moe_experts(h, gu, dn, idx, wgt, want, 0, assign=assign, identity=True)
        got = torch.full((T, H), 0.5, device=DEV)
        K().moe_experts(h.to(DEV), gu.to(DEV), dn.to(DEV), idx.to(DEV), wgt.to(DEV), got, 0, assign=assign, identity=True)
        assert close(got, want, 3e-5 if dtype == "float32" else 2.5e-2)
    only = torch.full((T, top), E, dtype=torch.int32)                             # no pair in any product
    got = torch.empty((T, H), device=DEV)
    K().moe_experts(h.to(DEV), gu.to(DEV), dn.to(DEV), only.to(DEV), wgt.to(DEV), got, 0, assign=True, identity=True)
    assert close(got, h.float() * wgt.sum(1, keepdim=True), 1e-5)


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
        # in bfloat16 a row whose router scores two experts or groups nearly alike may take the other one; such rows are
        # rare and the 32-bit runs compare every row sharply
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
    agrees(run_tail_one_by_one(m, toks, 70), want, dtype, "tail")            # across a page's border and the temperature's steps
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
def test_long_prompts_are_cut_into_segments(dtype):
    """A prompt of several segments, beside a short one, whole, as two long portions, and with its last tokens decoded."""
    cfg = CONFIGS["A"]
    toks, short = random_tokens(cfg["vocab"], 700, seed=15), random_tokens(cfg["vocab"], 20, seed=16)
    m = model_of("A", dtype)
    want = plain_logits("A", toks, dtype)
    agrees(run_whole(m, toks), want, dtype, "whole")
    agrees(run_in_pieces(m, [toks], [[80, 640]])[0], want, dtype, "portions")
    got = run_batched(m, [short, toks], [15, 690])
    agrees(got[1], want, dtype, "batch")
    agrees(got[0], plain_logits("A", short, dtype), dtype, "the short one")


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
def test_long_decoding(dtype):
    cfg = CONFIGS["A"]
    toks = random_tokens(cfg["vocab"], 300, seed=9)
    agrees(run_tail_one_by_one(model_of("A", dtype), toks, 297), plain_logits("A", toks, dtype), dtype)


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
        assert e.median() < 2e-2 and int((e > 0.1).sum()) <= 5, (float(e.median()), float(e.max()))


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
        assert off <= (0 if dtype == "float32" else 1)              # (a close call between experts may fall the other way)
    assert lm.model.cache.slots.held == 0
    again = lm.generate(prompts[:2], temperature=0, repeat_penalty=1.0, max_tokens=12)     # on used slots, pages and states
    if dtype == "float32":
        assert [r.tokens for r in again] == [r.tokens for r in got[:2]]


def test_decode_steps_are_recorded():
    lm = cima_b200.load(folder("A", sharp=False), dtype="bfloat16", max_tokens=1024, verbose=False)
    assert lm.model.graph_safe and lm.stepper.use_graphs


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
