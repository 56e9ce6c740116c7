"""The Gudarax decoder without a GPU: its configuration, the plain implementation's mechanisms against other statements of
the same mathematics, and the package's host logic (cache, rings of pages, states, steps, generation) on the CPU stand-in
kernels against the plain implementation."""
import copy
import math

import pytest
import torch

import cima_b200
from cima_b200.cache import CapacityError
from cima_b200.config import ConfigError, GudaraxConfig, lookup_architecture
from cima_b200.engine import StepEntry, build_plan
from gudarax_cases import CONFIGS, G_A, attention, config, cpu_model, plain_weights, row_errors
from gudarax_plain import (plain_attention, plain_delta, plain_delta_inputs, plain_delta_rule, plain_dense_ff, plain_embedding, plain_forward,
                           plain_gelu_tanh, plain_latent_attention, plain_moe, plain_rms, plain_route, plain_side_input, plain_silu, plain_slopes,
                           plain_taps, plain_visible)
from helpers import random_tokens, run_batched, run_in_pieces, run_tail_one_by_one, run_whole

TOL = 2e-4
D = torch.float64


# ------------------------------------------------------------------------------------------- configuration
def test_configuration_round_trip_and_plan():
    for cfg in CONFIGS.values():
        entry = lookup_architecture(cfg)
        typed = entry.parse(cfg)
        assert isinstance(typed, GudaraxConfig)
        assert GudaraxConfig.from_dict(typed.to_dict()) == typed
        plan = build_plan(entry.spec(typed))
        assert {"embed", "pos", "side.embed", "final.norm", "head"} <= set(plan)
    plan = build_plan(GudaraxConfig.from_dict(G_A).model_spec())
    assert plan["pos"].shape == (640, 96) and plan["side.embed"].shape == (300, 60)
    assert plan["l0.mix.dq"].shape == (28, 96) and plan["l0.mix.uq"].shape == (72, 28) and plan["l0.mix.dkv"].shape == (40, 96)
    assert plan["l0.mix.uk"].shape == (72, 40) and plan["l0.mix.uv"].shape == (60, 40) and plan["l0.mix.g"].shape == (60, 96)
    assert plan["l1.mix.q.b"].shape == (96,) and plan["l1.mix.q.norm"].shape == (96,) and plan["l1.mix.k.norm"].shape == (48,)
    assert plan["l1.mix.v"].shape == (32, 96) and plan["l1.mix.o"].shape == (96, 64)
    assert "l1.mix.vmix" not in plan and plan["l3.mix.vmix"].shape == () and "l4.mix.vmix" not in plan       # the first one mixes nothing in
    assert plan["l2.mix.a"].shape == (4, 96) and plan["l2.mix.dt_bias"].shape == (4,) and plan["l2.mix.k.conv"].shape == (32, 3)
    assert plan["l2.mix.norm"].shape == (24,) and plan["l2.mix.g"].shape == (96, 96)
    assert "l2.norm2" not in plan and "l2.mlp.router" not in plan and plan["l2.side.gate"].shape == (12, 96)     # no feed-forward
    assert plan["l0.mlp.e4.down"].shape == (96, 32) and "l0.mlp.e0.gate" not in plan and plan["l1.mlp.gate"].shape == (72, 96)


def test_sizes_that_are_left_out_take_their_usual_values():
    cfg = copy.deepcopy(G_A)
    for k in ("vdim", "scale", "kv_heads", "v_mix", "mask"):
        cfg["layers"][1]["mixer"].pop(k)
    a = GudaraxConfig.from_dict(cfg).layers[1].attention
    assert (a.vdim, a.kv_heads, a.window, a.v_mix) == (24, 4, 0, False) and a.scale == 24 ** -0.5


@pytest.mark.parametrize("change,word", [
    (lambda c: c.update(architecture="Other"), "architecture"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c["token_side"].update(dim=0), "dim"),
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=0), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(scale=-1.0), "scale"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=24), "v_mix"),
    (lambda c: c["layers"][2]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][3]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "kind"),
])
def test_configuration_refuses(change, word):
    cfg = copy.deepcopy(G_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        GudaraxConfig.from_dict(cfg)
    assert word in str(e.value)


# ------------------------------------------------------------------------------------------- the plain mechanisms
def test_plain_window_and_slopes():
    assert plain_visible(5, 3) == [3, 4, 5] and plain_visible(1, 3) == [0, 1] and plain_visible(4, 0) == [0, 1, 2, 3, 4] and plain_visible(7, 1) == [7]
    assert plain_slopes(8) == [0.5 ** h for h in range(1, 9)] and plain_slopes(2) == [2.0 ** -4, 2.0 ** -8]
    assert plain_slopes(3)[0] == 2.0 ** (-8.0 / 3.0)


def test_plain_attention_written_out_for_one_row():
    torch.manual_seed(1)
    m = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "scale": 0.7, "mask": {"size": 4}, "v_mix": True}
    W = {}
    for n, r in (("q", 24), ("k", 12), ("v", 6)):
        W[n], W[n + ".b"] = torch.randn(r, 10, dtype=D), torch.randn(r, dtype=D)
    W.update({"q.norm": torch.rand(24, dtype=D) + 0.5, "k.norm": torch.rand(12, dtype=D) + 0.5, "vmix": torch.tensor(0.3, dtype=D),
              "o": torch.randn(10, 12, dtype=D)})
    h, first = torch.randn(7, 10, dtype=D), torch.randn(7, 6, dtype=D)
    got, own = plain_attention(h, W, m, 1e-5, first)
    i, rows = 5, []
    q = W["q"] @ h[i] + W["q.b"]
    q = q / math.sqrt(float((q * q).sum()) / 24 + 1e-5) * W["q.norm"]                     # all heads at once
    for a in range(4):
        g, e, vs = a // 2, [], []
        for j in range(2, i + 1):                                                        # itself and the three before it
            k = W["k"] @ h[j] + W["k.b"]
            k = (k / math.sqrt(float((k * k).sum()) / 12 + 1e-5) * W["k.norm"])[g * 6:g * 6 + 6]
            e.append(math.exp(float(q[a * 6:a * 6 + 6] @ k) * 0.7 - 4.0 ** -(a + 1) * (i - j)))
            vs.append((0.7 * (W["v"] @ h[j] + W["v.b"]) + 0.3 * first[j])[g * 3:g * 3 + 3])
        rows.append(sum(x / sum(e) * v for x, v in zip(e, vs)))
    assert torch.allclose(got[i], W["o"] @ torch.cat(rows))
    assert torch.allclose(own, h @ W["v"].T + W["v.b"])                                   # what the first one hands on is not mixed
    alone, _ = plain_attention(h, W, dict(m, v_mix=False), 1e-5, first)
    assert torch.allclose(alone, plain_attention(h, dict(W, vmix=torch.tensor(0.0, dtype=D)), m, 1e-5, first)[0])


def test_plain_latent_attention_in_the_latents_space():
    """The same with the queries moved into the latents' space: no key and no value is ever built."""
    torch.manual_seed(2)
    m = {"heads": 3, "dim": 5, "vdim": 4, "kv_rank": 7, "q_rank": 6, "scale": 0.8}
    W = {"dq": torch.randn(6, 9, dtype=D), "dq.norm": torch.rand(6, dtype=D) + 0.5, "uq": torch.randn(15, 6, dtype=D), "dkv": torch.randn(7, 9, dtype=D),
         "dkv.norm": torch.rand(7, dtype=D) + 0.5, "uk": torch.randn(15, 7, dtype=D), "uv": torch.randn(12, 7, dtype=D), "g": torch.randn(12, 9, dtype=D),
         "o": torch.randn(9, 12, dtype=D)}
    h = torch.randn(8, 9, dtype=D)
    got = plain_latent_attention(h, W, m, 1e-6)
    q = (plain_rms(h @ W["dq"].T, 1e-6) * W["dq.norm"]) @ W["uq"].T
    c = plain_rms(h @ W["dkv"].T, 1e-6) * W["dkv.norm"]
    for t in range(8):
        heads = []
        for a in range(3):
            moved = W["uk"][a * 5:a * 5 + 5].T @ q[t, a * 5:a * 5 + 5]
            p = torch.softmax((c[:t + 1] @ moved) * 0.8, 0)
            heads.append(W["uv"][a * 4:a * 4 + 4] @ (p @ c[:t + 1]))
        assert torch.allclose(got[t], W["o"] @ (torch.cat(heads) / (1.0 + torch.exp(-(W["g"] @ h[t])))))


def test_plain_delta_rule_stores_and_replaces():
    """A key written twice with beta 1 and no decay holds the second value; the read-out sees the token's own write; a decay of g
    leaves g times what another key held."""
    e = torch.eye(3, dtype=D)
    k = torch.stack([e[0], e[1], e[0]])[:, None]
    v = torch.tensor([[1.0, 2.0], [5.0, 6.0], [-3.0, 4.0]], dtype=D)[:, None]
    one = torch.ones(3, 1, dtype=D)
    out = plain_delta_rule(k, k, v, one, one)
    assert torch.equal(out[:, 0], v[:, 0])                                                # each token reads its own write
    q = torch.stack([e[1], e[0], e[1]])[:, None]
    assert torch.equal(plain_delta_rule(q, k, v, one, one)[:, 0], torch.stack([torch.zeros(2, dtype=D), v[0, 0], v[1, 0]]))
    half = plain_delta_rule(q, k, v, one, one * 0.5)[:, 0]
    assert torch.allclose(half, torch.stack([torch.zeros(2, dtype=D), 0.5 * v[0, 0], 0.5 * v[1, 0]]))


def test_plain_delta_equals_its_matrix_form():
    """S_t = g_t (I - beta_t k k^T) S_(t-1) + beta_t k v^T."""
    torch.manual_seed(3)
    m = {"heads": 4, "kv_heads": 2, "dim": 5, "vdim": 3, "conv": 3}
    W = {"q": torch.randn(10, 8, dtype=D), "k": torch.randn(10, 8, dtype=D), "v": torch.randn(12, 8, dtype=D), "b": torch.randn(4, 8, dtype=D),
         "a": torch.randn(4, 8, dtype=D), "A_log": torch.randn(4, dtype=D), "dt_bias": torch.randn(4, dtype=D), "norm": torch.rand(3, dtype=D) + 0.5,
         "g": torch.randn(12, 8, dtype=D), "o": torch.randn(8, 12, dtype=D)}
    W.update({n + ".conv": torch.randn(W[n].shape[0], 3, dtype=D) for n in ("q", "k", "v")})
    h = torch.randn(9, 8, dtype=D)
    q, k, v, beta, g = plain_delta_inputs(h, W, m)
    assert torch.allclose(k.norm(dim=-1), torch.ones(9, 2, dtype=D), atol=1e-3) and torch.allclose(q.norm(dim=-1), torch.full((9, 2), 5 ** -0.5, dtype=D), atol=1e-3)
    assert torch.allclose(g, torch.sigmoid(-(h @ W["a"].T + W["dt_bias"])) ** torch.exp(W["A_log"]))         # exp(-r softplus(z)) = sigmoid(-z)^r
    out = torch.zeros(9, 4, 3, dtype=D)
    for a in range(4):
        S = torch.zeros(5, 3, dtype=D)
        for t in range(9):
            kk = k[t, a // 2]
            S = g[t, a] * (torch.eye(5, dtype=D) - beta[t, a] * torch.outer(kk, kk)) @ S + beta[t, a] * torch.outer(kk, v[t, a])
            out[t, a] = S.T @ q[t, a // 2]
    assert torch.allclose(plain_delta_rule(q, k, v, beta, g), out)
    y = out / torch.sqrt((out * out).mean(-1, keepdim=True) + 1e-5) * W["norm"]
    assert torch.allclose(plain_delta(h, W, m, 1e-5), (y.reshape(9, 12) * plain_silu(h @ W["g"].T)) @ W["o"].T)


def test_plain_taps_reach_back_from_the_last_column():
    z = torch.arange(1.0, 6.0, dtype=D)[:, None]
    assert torch.equal(plain_taps(z, torch.tensor([[100.0, 10.0, 1.0]], dtype=D))[:, 0], torch.tensor([1.0, 12.0, 123.0, 234.0, 345.0], dtype=D))
    assert torch.equal(plain_taps(z, torch.tensor([[2.0]], dtype=D)), 2 * z)


def test_plain_feed_forwards_and_token_input():
    z = torch.linspace(-4, 4, 33, dtype=D)
    assert torch.allclose(plain_gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert plain_route(torch.tensor([0.1, 0.7, 0.3, 0.6]), 3) == [1, 3, 2]
    torch.manual_seed(4)
    W = {"router": torch.randn(3, 5, dtype=D)}
    for e in range(3):
        W.update({f"e{e}.up": torch.randn(4, 5, dtype=D), f"e{e}.down": torch.randn(5, 4, dtype=D)})
    h = torch.randn(9, 5, dtype=D)
    got = plain_moe(h, W, {"experts": 3, "top": 2})
    for t in range(9):
        s = 1.0 / (1.0 + torch.exp(-(W["router"] @ h[t])))
        want = torch.zeros(5, dtype=D)
        for e in s.topk(2).indices.tolist():           # the square of ReLU is of degree two: a weight on the input counts squared
            want += s[e] ** 2 * (W[f"e{e}.down"] @ torch.relu(W[f"e{e}.up"] @ h[t]) ** 2)
        assert torch.allclose(got[t], want)
    x, table = torch.randn(4, 6, dtype=D), torch.randn(10, 8, dtype=D)
    S = {"gate": torch.randn(2, 6, dtype=D), "proj": torch.randn(6, 2, dtype=D), "norm": torch.rand(6, dtype=D)}
    y = plain_side_input(x, [3, 3, 9, 0], table, 2, 2, S, 1e-5)
    row = S["proj"] @ (plain_gelu_tanh(S["gate"] @ x[2]) * table[9, 4:6])
    assert torch.allclose(y[2], row / math.sqrt(float((row * row).mean()) + 1e-5) * S["norm"])
    assert torch.allclose(plain_embedding([2, 2], table, x[:, :1].expand(4, 8), 3.0)[1], 3.0 * table[2] + x[1, 0])
    assert torch.allclose(plain_dense_ff(h, {"gate": W["e0.up"], "up": W["e1.up"], "down": W["e2.down"]})[0],
                          W["e2.down"] @ (torch.nn.functional.silu(W["e0.up"] @ h[0]) * (W["e1.up"] @ h[0])))


# ------------------------------------------------------------------------------------------- host logic on the stand-ins
@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_cutting_on_the_cpu(name):
    cfg, W = plain_weights(name)
    toks, other = random_tokens(cfg["vocab"], 150, seed=3), random_tokens(cfg["vocab"], 70, seed=4)
    want, want2 = plain_forward(cfg, W, toks), plain_forward(cfg, W, other)
    m = cpu_model(name)
    assert row_errors(run_whole(m, toks), want).max() < TOL
    assert row_errors(run_tail_one_by_one(m, toks[:110], 50), want[:110]).max() < TOL
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
    kept = {(g.request.n_kv_heads, g.request.head_dim, g.request.window, g.request.planes): g.ring_pages for g in m.cache.groups}
    assert kept == {(1, 40, 0, 1): 0, (2, 32, 40, 2): 2, (2, 48, 100, 2): 3, (1, 32, 0, 2): 0}
    state = {n: tuple(t.shape[1:]) for n, t in m.cache.state.items() if not n.startswith("sampler")}
    assert state == {"delta.2": (4, 16, 24), "short_conv.2": (2, 160)}
    assert m.cache.state["delta.2"].dtype is torch.float32


def test_a_step_leaves_nothing_for_the_next_one():
    """The values that mixing layers share belong to one step's tokens."""
    from cima_b200.engine.batch import build_batch
    m = cpu_model("A")
    (slot,) = m.cache.open(1)
    m.cache.reserve(slot, 5)
    m.cache.flush()
    b = build_batch([StepEntry(slot, [1, 2, 3, 4, 5], [4])], [0], 300, "cpu")
    m.forward(b)
    assert b.carried == {}
    m.cache.close([slot])


def test_positions_end_where_the_table_ends():
    cfg, W = plain_weights("B")
    m = cpu_model("B", max_tokens=1024)
    toks = random_tokens(cfg["vocab"], 300, seed=1)
    assert row_errors(run_tail_one_by_one(m, toks, 3), plain_forward(cfg, W, toks)).max() < TOL       # up to the last position
    (slot,) = m.cache.open(1)
    with pytest.raises(CapacityError):
        m.step([StepEntry(slot, toks + [1], [300])])
    m.cache.close([slot])


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


def test_names_that_nothing_reads_are_let_through(tmp_path):
    """The first mixing layer's number and the norm in front of an absent feed-forward may be stored; another name may not."""
    from safetensors.torch import load_file, save_file
    from cima_b200.weights import load_tensors
    from cima_b200.weights.loader import WeightError
    from cima_b200.engine.model import Model
    from cima_b200.parts import Runtime
    cima_b200.write_random_model(str(tmp_path), G_A, seed=1)
    path = str(tmp_path / "model.safetensors")
    t = load_file(path)
    t.update({"l1.mix.vmix": torch.tensor(0.5), "l2.norm2": torch.ones(96)})
    save_file(t, path)
    spec = GudaraxConfig.from_dict(G_A).model_spec()
    m = Model(spec, Runtime(kernels=None, dtype=torch.float32, device="cpu"))
    assert set(load_tensors(str(tmp_path), m.plan(), ignore=m.ignorable())) == set(m.plan())
    t["l2.mix.sink"] = torch.ones(4)
    save_file(t, path)
    with pytest.raises(WeightError, match="l2.mix.sink"):
        load_tensors(str(tmp_path), m.plan(), ignore=m.ignorable())


# ------------------------------------------------------------------------------------------- the weights show a fault
def test_sharp_maps_rest_on_single_far_keys():
    cfg, W = plain_weights("C")
    maps = {}
    plain_forward(cfg, W, random_tokens(cfg["vocab"], 260, seed=5), attention_out=maps)
    for layer, P in maps.items():
        top, at = P[:, 130:].max(dim=-1)
        window = cfg["layers"][layer]["mixer"].get("mask", {}).get("size", 10 ** 6)
        far = (top > 0.3) & (torch.arange(130, 260)[None, :] - at > min(64, window // 2))
        assert int(far.sum()) >= 15, (layer, int(far.sum()))       # rows that a key far back carries


def test_a_windows_edges_carry_rows():
    cfg, W = plain_weights("C")
    maps = {}
    plain_forward(cfg, W, random_tokens(cfg["vocab"], 300, seed=6), attention_out=maps)
    for layer in (0, 3, 5):
        w = cfg["layers"][layer]["mixer"]["mask"]["size"]
        P = maps[layer]
        oldest = torch.stack([P[:, i, i - w + 1] for i in range(w, 300)])          # the last position inside the window
        assert float(oldest.max()) > 0.2, (layer, float(oldest.max()))
        assert all(float(P[:, i, i - w].max()) == 0.0 for i in range(w, 300))


@pytest.mark.parametrize("name,tensor,change", [
    ("A", "pos", lambda t: t * 0.0), ("A", "side.embed", lambda t: t.flip(1)), ("A", "l2.side.norm", lambda t: t * 0.0), ("A", "l0.mix.g", lambda t: t * 0.0),
    ("A", "l3.mix.vmix", lambda t: t * 0.0), ("A", "l1.mix.q.b", lambda t: t * 0.0), ("A", "l1.mix.k.b", lambda t: t * 0.0), ("A", "l1.mix.v.b", lambda t: t * 0.0),
    ("A", "l3.mix.q.norm", lambda t: t.flip(0)), ("A", "l2.mix.dt_bias", lambda t: t + 2.0), ("A", "l2.mix.A_log", lambda t: t.flip(0)),
    ("A", "l2.mix.k.conv", lambda t: t.flip(1)), ("A", "l2.mix.g", lambda t: t * 0.0), ("A", "l0.mix.dq.norm", lambda t: t.flip(0) * 1.5)])
def test_a_tensor_left_out_shows(name, tensor, change):
    cfg, W = plain_weights(name)
    toks = random_tokens(cfg["vocab"], 40, seed=13)
    base = plain_forward(cfg, W, toks)
    assert row_errors(plain_forward(cfg, dict(W, **{tensor: change(W[tensor])}), toks), base).max() > 0.02


@pytest.mark.parametrize("edit", [lambda c: c["layers"][1]["mixer"]["mask"].update(size=41), lambda c: c["layers"][1]["mixer"]["mask"].update(size=39),
                                  lambda c: c["layers"][3]["mixer"].update(v_mix=False), lambda c: c["embedding"].update(scale=1.9),
                                  lambda c: c["layers"][0]["mlp"]["router"].update(top=1), lambda c: c["layers"][4]["mixer"].update(mask={"size": 60})])
def test_a_constant_that_is_off_shows(edit):
    cfg, W = plain_weights("A")
    toks = random_tokens(cfg["vocab"], 120, seed=14)
    other = copy.deepcopy(cfg)
    edit(other)
    assert row_errors(plain_forward(other, W, toks), plain_forward(cfg, W, toks)).max() > 0.02


def test_mixed_values_between_heads_padded_differently():
    """The mixing layers' heads are padded to other sizes in the cache than the first one's."""
    import tempfile
    from gudarax_cases import write_folder
    from gudarax_plain import read_folder
    from cima_b200.engine import load_model
    from reference_kernels import ReferenceKernels
    cfg = config(90, 32, 200, 1e-5, 1.0, 3, [attention(2, 2, 8, 20, 0.9, 0, True, None), attention(4, 2, 60, 20, 0.4, 9, True, None),
                                             attention(2, 2, 33, 20, 0.4, 70, True, None)])
    d = write_folder(tempfile.mkdtemp(), cfg, 3)
    c, W = read_folder(d)
    m = load_model(d, dtype="float32", max_tokens=512, device="cpu", kernels=ReferenceKernels(), verbose=False)
    assert [b.mixer.hd for b in m.blocks] == [32, 64, 48]
    toks = random_tokens(90, 100, seed=2)
    want = plain_forward(c, W, toks)
    assert row_errors(run_whole(m, toks), want).max() < TOL and row_errors(run_tail_one_by_one(m, toks, 40), want).max() < TOL
