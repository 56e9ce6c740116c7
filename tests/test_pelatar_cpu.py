"""The Pelatar decoder without a GPU: its configuration, the plain implementation's mechanisms against other statements of
the same mathematics, and the package's host logic (cache, pages, states, steps, generation) on the CPU stand-in kernels
against the plain implementation."""
import copy
import math

import pytest
import torch

import cima_b200
from cima_b200.config import ConfigError, PelatarConfig, lookup_architecture
from cima_b200.engine import StepEntry, build_plan
from pelatar_cases import CONFIGS, P_A, P_B, P_C, cpu_model, plain_weights, row_errors
from pelatar_plain import (plain_attention, plain_dense_ff, plain_forward, plain_gelu_tanh, plain_gla_decays, plain_gla_memory,
                           plain_keys_values, plain_log_sigmoid, plain_mlstm_gates, plain_mlstm_memory, plain_moe,
                           plain_query_temperature, plain_rms, plain_route, plain_silu, plain_sink_softmax)
from helpers import random_tokens, run_batched, run_in_pieces, run_tail_one_by_one, run_whole

TOL = 2e-4
D = torch.float64


# ------------------------------------------------------------------------------------------- configuration
def test_configuration_round_trip_and_plan():
    for cfg in CONFIGS.values():
        entry = lookup_architecture(cfg)
        typed = entry.parse(cfg)
        assert isinstance(typed, PelatarConfig)
        assert PelatarConfig.from_dict(typed.to_dict()) == typed
        plan = build_plan(entry.spec(typed))
        assert "embed" in plan and "final.norm" in plan and "head" not in plan          # the table is the head
    plan = build_plan(PelatarConfig.from_dict(P_A).model_spec())
    assert plan["l0.mix.q"].shape == (72, 96) and plan["l0.mix.v"].shape == (120, 96) and plan["l0.mix.a1"].shape == (8, 96)
    assert plan["l0.mix.a2"].shape == (72, 8) and plan["l0.mix.a2.b"].shape == (72,) and plan["l0.mix.norm"].shape == (40,)
    assert plan["l1.mix.q"].shape == (96, 96) and plan["l1.mix.k"].shape == (48, 96) and plan["l1.mix.v"].shape == (32, 96)
    assert plan["l1.mix.g"].shape == (64, 96) and plan["l1.mix.o"].shape == (96, 64) and plan["l1.mix.sink"].shape == (4,)
    assert "l2.mix.k" not in plan and "l2.mix.v" not in plan and plan["l2.mix.g"].shape == (64, 96)      # reads layer 1's
    assert plan["l3.mix.i"].shape == (2, 96) and plan["l3.mix.f.b"].shape == (2,) and plan["l3.mix.norm"].shape == (48,)
    assert "l3.norm2" not in plan and "l3.mlp.gate" not in plan                          # a layer without feed-forward
    assert plan["l1.mlp.router"].shape == (8, 96) and plan["l1.mlp.correction"].shape == (8,) and "l1.mlp.e5.up" not in plan
    assert plan["l1.mlp.e4.down"].shape == (96, 32) and plan["l0.mlp.gate"].shape == (72, 96)


def test_the_rank_and_what_is_stored_are_read_off_the_tensors():
    cfg = copy.deepcopy(P_A)
    del cfg["layers"][0]["mixer"]["rank"]
    assert PelatarConfig.from_dict(cfg).layers[0].memory.rank == 16
    typed = PelatarConfig.from_dict(cfg, shapes={"l0.mix.a1": (5, 96), "l1.mix.sink": (4,)})
    assert typed.layers[0].memory.rank == 5 and typed.layers[1].attention.sink and not typed.layers[2].attention.sink
    assert not typed.layers[1].moe.correction


@pytest.mark.parametrize("change,word", [
    (lambda c: c.update(architecture="Other"), "architecture"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=24), "kv_from"),
    (lambda c: c["layers"][0]["mixer"].update(tau=-1.0), "tau"),
    (lambda c: c["layers"][3]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "kind"),
])
def test_configuration_refuses(change, word):
    cfg = copy.deepcopy(P_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        PelatarConfig.from_dict(cfg)
    assert word in str(e.value)


# ------------------------------------------------------------------------------------------- the plain mechanisms
def test_plain_temperature_steps_where_a_block_of_positions_is_full():
    f = lambda p: plain_query_temperature(p, 0.3, 8)
    assert f(0) == 1.0 and f(6) == 1.0                            # floor(7 / 8) = 0
    assert f(7) == 1.0 + 0.3 * math.log(2.0) == f(14) and f(15) == 1.0 + 0.3 * math.log(3.0)
    assert plain_query_temperature(0, 0.5, 1) == 1.0 + 0.5 * math.log(2.0)


def test_plain_sink_is_one_more_column_that_carries_nothing():
    torch.manual_seed(0)
    for sink in (-40.0, -1.0, 0.0, 3.0, 40.0):
        s = torch.randn(6, dtype=D) * 3
        p = plain_sink_softmax(s, torch.tensor(sink, dtype=D))
        assert torch.allclose(p, torch.softmax(torch.cat([s, torch.tensor([sink], dtype=D)]), 0)[:-1])


def test_plain_attention_written_out_for_one_row():
    torch.manual_seed(1)
    m = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "scale": 0.7, "q_temp": {"coef": 0.5, "every": 3}}
    W = {k: torch.randn(r, 10, dtype=D) for k, r in (("q", 24), ("k", 12), ("v", 6), ("g", 12))}
    W.update(o=torch.randn(10, 12, dtype=D), sink=torch.tensor([0.5, -1.0, 2.0, 0.0], dtype=D))
    h = torch.randn(7, 10, dtype=D)
    got = plain_attention(h, W, m, 1e-5)
    i, rows = 5, []
    for a in range(4):
        g = a // 2
        q = W["q"][a * 6:a * 6 + 6] @ h[i]
        q = q / math.sqrt(float((q * q).mean()) + 1e-5) * (1.0 + 0.5 * math.log(3.0))      # (5 + 1) / 3 = 2 full blocks
        e = []
        for j in range(i + 1):
            k = W["k"][g * 6:g * 6 + 6] @ h[j]
            e.append(math.exp(float(q @ k) / math.sqrt(float((k * k).mean()) + 1e-5) * 0.7))
        den = sum(e) + math.exp(float(W["sink"][a]))
        rows.append(sum(e[j] / den * (W["v"][g * 3:g * 3 + 3] @ h[j]) for j in range(i + 1)))
    assert torch.allclose(got[i], W["o"] @ (torch.cat(rows) / (1.0 + torch.exp(-(W["g"] @ h[i])))))
    # another layer's keys and values are taken as they are stored
    k, v = plain_keys_values(h, W, m, 1e-5)
    assert torch.allclose(k.pow(2).mean(-1), torch.ones(7, 2, dtype=D), atol=1e-4)
    assert torch.allclose(plain_attention(h, {n: t for n, t in W.items() if n not in ("k", "v")}, m, 1e-5, (k, v)), got)


def test_plain_mlstm_equals_its_unrolled_sum():
    """Without the running maximum: with F the sum of the log forget gates, token s counts e^(F_t - F_s + i_s) at t; the
    maximum cancels but for the denominator's lower bound (1 on this scale) and the small constant."""
    torch.manual_seed(2)
    T, H, dim, vdim = 12, 2, 5, 3
    q, k, v = torch.randn(T, H, dim, dtype=D), torch.randn(T, H, dim, dtype=D), torch.randn(T, H, vdim, dtype=D)
    i, f = torch.randn(T, H, dtype=D) * 3, plain_log_sigmoid(torch.randn(T, H, dtype=D) * 2 + 1)
    got = plain_mlstm_memory(q, k, v, i, f)
    F = torch.cumsum(f, 0)
    for t in range(T):
        for h in range(H):
            w = [math.exp(float(F[t, h] - F[s, h] + i[s, h])) * float(k[s, h] @ q[t, h]) for s in range(t + 1)]
            m = max([float(F[t, h])] + [float(F[t, h] - F[s, h] + i[s, h]) for s in range(t + 1)])        # m starts at 0, not at -inf
            den = max(abs(sum(w)), 1.0) + 1e-6 * math.exp(m)
            assert torch.allclose(got[t, h], sum(w[s] * v[s, h] for s in range(t + 1)) / den)


def test_plain_mlstm_gates_are_capped():
    W = {"i": torch.eye(2, dtype=D), "f": torch.eye(2, dtype=D), "i.b": torch.tensor([0.5, 0.0], dtype=D), "f.b": torch.zeros(2, dtype=D)}
    i, f = plain_mlstm_gates(torch.tensor([[1e4, -1e4], [0.1, 0.2]], dtype=D), W, 4.0)
    assert torch.allclose(i[0], torch.tensor([4.0, -4.0], dtype=D))
    assert torch.allclose(f[0], torch.log(torch.sigmoid(torch.tensor([4.0, -4.0], dtype=D))))
    assert abs(float(i[1, 0]) - 4.0 * math.tanh(0.6 / 4.0)) < 1e-15
    z = torch.tensor([-800.0, -5.0, 0.0, 5.0, 800.0], dtype=D)
    assert torch.allclose(plain_log_sigmoid(z), torch.nn.functional.logsigmoid(z))


def test_plain_gla_equals_its_unrolled_sum():
    torch.manual_seed(3)
    T, H, dim, vdim = 10, 2, 4, 3
    q, k, v = torch.randn(T, H, dim, dtype=D), torch.randn(T, H, dim, dtype=D), torch.randn(T, H, vdim, dtype=D)
    a = torch.rand(T, H, dim, dtype=D)
    got = plain_gla_memory(q, k, v, a)
    for t in range(T):
        want = torch.zeros(H, vdim, dtype=D)
        for s in range(t + 1):
            decay = torch.ones(H, dim, dtype=D)
            for r in range(s + 1, t + 1):
                decay = decay * a[r]
            want += (q[t] * decay * k[s]).sum(-1, keepdim=True) * v[s]
        assert torch.allclose(got[t], want)
    W = {"a1": torch.randn(2, 5, dtype=D), "a2": torch.randn(3, 2, dtype=D), "a2.b": torch.randn(3, dtype=D)}
    h = torch.randn(4, 5, dtype=D)
    z = h @ (W["a2"] @ W["a1"]).T + W["a2.b"]
    assert torch.allclose(plain_gla_decays(h, W, 7.0), torch.sigmoid(z) ** (1.0 / 7.0))


def test_plain_feed_forwards():
    z = torch.linspace(-4, 4, 33, dtype=D)
    assert torch.allclose(plain_gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    # groups are compared by their best choice score, negative ones included; the weights leave the correction out
    s = torch.tensor([0.1, 0.3, 0.2, 0.05, 0.25, 0.1], dtype=D)
    assert plain_route(s, torch.zeros(6, dtype=D), 2, 3, 1) == [1, 0]                     # group (0, 1) holds the best expert
    assert plain_route(s, torch.tensor([0, -1.0, 0, 0, 0, 0], dtype=D), 2, 3, 1) == [4, 5]
    assert plain_route(s - 5.0, torch.zeros(6, dtype=D), 3, 3, 2) == [1, 4, 0]             # all negative: still only the kept groups'
    torch.manual_seed(4)
    mlp = {"router": {"experts": 3, "identity": 1, "top": 2, "groups": {"count": 2, "keep": 1}}}
    W = {"router": torch.randn(4, 5, dtype=D), "correction": torch.randn(4, dtype=D) * 0.3}
    for e in range(3):
        W.update({f"e{e}.gate": torch.randn(2, 5, dtype=D), f"e{e}.up": torch.randn(2, 5, dtype=D), f"e{e}.down": torch.randn(5, 2, dtype=D)})
    h = torch.randn(9, 5, dtype=D)
    got, seen = plain_moe(h, W, mlp), set()
    for t in range(9):
        s = torch.softmax(W["router"] @ h[t], 0)
        c = s + W["correction"]
        group = 0 if float(c[:2].max()) > float(c[2:].max()) else 1
        seen.add(group)
        want = torch.zeros(5, dtype=D)
        for e in (2 * group, 2 * group + 1):                                             # two of the group's two
            out = h[t] if e == 3 else W[f"e{e}.down"] @ (plain_silu(W[f"e{e}.gate"] @ h[t]) * (W[f"e{e}.up"] @ h[t]))
            want += s[e] * out
        assert torch.allclose(got[t], want)
    assert seen == {0, 1}


def test_plain_layer_norms_what_it_adds_only():
    cfg, W = plain_weights("B")
    cfg = dict(cfg, layers=cfg["layers"][:2])
    toks = random_tokens(cfg["vocab"], 9, seed=1)
    _, streams = plain_forward(cfg, W, toks, return_layers=True)
    added = streams[1] - streams[0]                                # the second layer has no feed-forward
    y = added / W["l1.norm1"]
    assert torch.allclose(y.pow(2).mean(-1), torch.ones(9, dtype=D), atol=1e-3)            # a normed row, times the weight
    # scaling a sublayer's output product changes nothing (but for eps): the norm behind it takes the factor out
    W2 = dict(W)
    W2["l1.mix.o"] = W["l1.mix.o"] * 3.0
    assert torch.allclose(plain_forward(cfg, W2, toks), plain_forward(cfg, W, toks), atol=1e-3)


# ------------------------------------------------------------------------------------------- host logic on the stand-ins
@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_cutting_on_the_cpu(name):
    cfg, W = plain_weights(name)
    toks, other = random_tokens(cfg["vocab"], 150, seed=3), random_tokens(cfg["vocab"], 70, seed=4)
    want, want2 = plain_forward(cfg, W, toks), plain_forward(cfg, W, other)
    m = cpu_model(name)
    assert row_errors(run_whole(m, toks), want).max() < TOL
    assert row_errors(run_tail_one_by_one(m, toks[:90], 25), want[:90]).max() < TOL
    got = run_in_pieces(m, [toks, other], [[2, 4, 7, 64, 66, 140], [63, 65]])
    assert row_errors(got[0], want).max() < TOL and row_errors(got[1], want2).max() < TOL
    got = run_batched(m, [toks[:80], other[:9], other], [70, 3, 64])
    assert row_errors(got[0], want[:80]).max() < TOL and row_errors(got[1], want2[:9]).max() < TOL and row_errors(got[2], want2).max() < TOL
    m.cache.check()
    assert m.cache.slots.held == 0


def test_the_stream_after_every_layer():
    cfg, W = plain_weights("A")
    toks = random_tokens(cfg["vocab"], 30, seed=8)
    _, streams = plain_forward(cfg, W, toks, return_layers=True)
    m = cpu_model("A")
    (slot,) = m.cache.open(1)
    seen = []
    for blk in m.blocks:
        orig = blk.forward
        def wrapped(x, *a, _o=orig, **k):
            r = _o(x, *a, **k)
            seen.append(x.detach().double().clone())
            return r
        blk.forward = wrapped
    m.step([StepEntry(slot, toks, [len(toks) - 1])])
    m.cache.close([slot])
    assert len(seen) == len(cfg["layers"])
    for got, want in zip(seen, streams):
        assert float((got - want).abs().max()) < 2e-4 * float(want.abs().max())


def test_what_a_sequence_keeps():
    m = cpu_model("A")
    assert len(m.cache.groups) == 1 and len(m.cache.groups[0].layers) == 1        # two layers read the third's pages
    assert m.cache.groups[0].request.head_dim == 32 and m.cache.groups[0].request.window == 0
    state = {n: tuple(t.shape[1:]) for n, t in m.cache.state.items() if not n.startswith("sampler")}
    assert state == {"gated_linear_attention.0": (3, 24, 40), "mlstm.3": (2, 16, 24), "mlstm.3.n": (2, 16), "mlstm.3.m": (2,)}
    assert all(t.dtype is torch.float32 for n, t in m.cache.state.items() if n in state)


def test_reused_slots_pages_and_states_start_from_nothing():
    cfg, W = plain_weights("B")
    m = cpu_model("B", max_tokens=128, max_seqs=1)
    for seed in (1, 2, 3):
        toks = random_tokens(cfg["vocab"], 70, seed=seed)
        assert row_errors(run_tail_one_by_one(m, toks, 10), plain_forward(cfg, W, toks)).max() < TOL


def test_greedy_generation_on_the_cpu():
    from cima_b200 import LM
    cfg, W = plain_weights("B")
    lm = LM(cpu_model("B"), [], max_batch=4, pipeline=False, use_graphs=False)
    prompts = [random_tokens(cfg["vocab"], n, seed=20 + n) for n in (5, 1, 12)]
    got = lm.generate(prompts, temperature=0, repeat_penalty=1.0, max_tokens=6)
    for p, r in zip(prompts, got):
        seq = list(p)
        for t in r.tokens:
            lg = plain_forward(cfg, W, seq)[-1]
            assert lg[t] >= lg.max() - 1e-4
            seq.append(t)


def test_tensors_by_name_round_trip():
    for name in CONFIGS:
        m = cpu_model(name)
        sd = m.state_dict()
        cfg, W = plain_weights(name)
        assert set(sd) == set(W)
        for n, t in W.items():
            assert torch.equal(sd[n].double().reshape(t.shape), t), n


# ------------------------------------------------------------------------------------------- the weights show a fault
def test_sharp_maps_rest_on_single_far_keys():
    cfg, W = plain_weights("A")
    maps = {}
    plain_forward(cfg, W, random_tokens(cfg["vocab"], 200, seed=5), attention_out=maps)
    for layer, P in maps.items():
        top, at = P[:, 80:].max(dim=-1)
        far = (top > 0.4) & (torch.arange(80, 200)[None, :] - at > 64)
        assert int(far.sum()) >= 20, (layer, int(far.sum()))       # rows that a key more than a page back carries
        assert float((1.0 - P.sum(-1)).max()) > 0.2                # and rows of which the sink takes a part


@pytest.mark.parametrize("name,tensor,change", [("A", "l1.mix.sink", lambda t: t - 30.0), ("A", "l1.mix.g", lambda t: t * 0.0),
                                                ("A", "l1.mlp.correction", lambda t: t * 0.0), ("B", "l2.mix.a2.b", lambda t: t + 3.0),
                                                ("A", "l3.mix.f.b", lambda t: t - 3.0), ("A", "l3.mix.i.b", lambda t: t + 4.0)])
def test_a_tensor_left_out_shows(name, tensor, change):
    cfg, W = plain_weights(name)
    toks = random_tokens(cfg["vocab"], 40, seed=13)
    base = plain_forward(cfg, W, toks)
    assert row_errors(plain_forward(cfg, dict(W, **{tensor: change(W[tensor])}), toks), base).max() > 0.02


@pytest.mark.parametrize("edit", [lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=17), lambda c: c["layers"][1]["mixer"].pop("q_temp"),
                                  lambda c: c["layers"][0]["mixer"].update(tau=4.5), lambda c: c["layers"][3]["mixer"].update(gate_cap=3.0)])
def test_a_constant_that_is_off_shows(edit):
    cfg, W = plain_weights("A")
    toks = random_tokens(cfg["vocab"], 60, seed=14)
    other = copy.deepcopy(cfg)
    edit(other)
    assert row_errors(plain_forward(other, W, toks), plain_forward(cfg, W, toks)).max() > 0.02
