"""Pelatar configurations drawn at random (every size and constant that config.json gives, layer by layer, in any order of
the three mixers and the three feed-forwards) in cuttings drawn at random too (whole, a tail one by one, pieces, unequal
batches): in 32-bit against the plain implementation on weights that make attention sharp, and in bfloat16 against the
32-bit engine on a milder scale of the same configuration."""
import os
import random

import pytest
import torch

from cima_b200.engine import load_model
from pelatar_cases import attention, config, dense, gla, mlstm, moe, row_errors, write_folder
from pelatar_plain import plain_forward, read_folder
from helpers import random_tokens, run_batched, run_in_pieces, run_tail_one_by_one, run_whole

pytestmark = pytest.mark.gpu

SEEDS = list(range(int(os.environ.get("CIMA_RANDOM_CONFIGS", "8"))))


def draw_mlp(rng: random.Random):
    r = rng.random()
    if r < 0.2:
        return None
    if r < 0.5:
        return dense(rng.choice([8, 20, 33, 64, 96, 130]))
    count = rng.choice([1, 1, 2, 3, 4, 6])
    per = rng.choice([1, 2, 3, 4, 5])
    total = count * per
    identity = rng.randint(0, total - 1)
    keep = rng.randint(1, count)
    groups = None if count == 1 and rng.random() < 0.5 else (count, keep)
    return moe(total - identity, identity, rng.randint(1, min(keep * per, 5)), rng.choice([8, 16, 24, 40, 64]), groups)


def draw_config(rng: random.Random) -> dict:
    width = rng.choice([16, 24, 25, 32, 48, 64, 80, 100, 128, 192, 320])            # some are no multiple of 8
    layers, own = [], []
    for i in range(rng.randint(1, 6)):
        r = rng.random()
        if r < 0.45:
            temp = (rng.choice([0.1, 0.3, 0.6]), rng.choice([1, 7, 64, 128, 4096])) if rng.random() < 0.8 else None
            src = rng.choice(own) if own and rng.random() < 0.5 else None
            if src is None:
                kv = rng.choice([1, 2, 3])
                sizes = (kv * rng.choice([1, 2, 4]), kv, rng.choice([8, 16, 20, 32, 48, 64, 80, 128]), rng.choice([8, 16, 24, 32, 64, 80, 96, 128]))
                own.append(i)
            else:
                m = layers[src]["mixer"]
                sizes = (m["heads"], m["kv_heads"], m["dim"], m["vdim"])
            layers.append(attention(*sizes, rng.choice([0.5, 1.0, 4.0]) * sizes[2] ** -0.5, temp, draw_mlp(rng), src))
        elif r < 0.72:
            layers.append(mlstm(rng.randint(1, 5), rng.choice([8, 16, 24, 32, 48, 64, 100, 136]), rng.choice([8, 20, 32, 64, 65, 96]),
                                rng.choice([2.0, 8.0, 15.0]), draw_mlp(rng)))
        else:
            layers.append(gla(rng.randint(1, 5), rng.choice([8, 16, 24, 32, 48, 64, 100, 136]), rng.choice([8, 20, 32, 64, 65, 96]),
                              rng.choice([1.0, 4.0, 16.0]), rng.choice([1, 4, 16, 24]), draw_mlp(rng)))
    return config(rng.choice([129, 333, 512, 1001]), width, rng.choice([1e-6, 1e-5, 3e-4]), layers)


@pytest.mark.parametrize("seed", SEEDS)
def test_random_configuration(seed, tmp_path):
    rng = random.Random(11000 + seed)
    cfg = draw_config(rng)
    folders = {kind: write_folder(str(tmp_path / kind), cfg, seed, sharp=kind == "sharp") for kind in ("sharp", "mild")}
    c, W = read_folder(folders["sharp"])
    n = rng.choice([40, 130, 300, 560])
    toks = random_tokens(cfg["vocab"], n, seed)
    want = plain_forward(c, W, toks)
    cuts = sorted(rng.sample(range(1, n), 3))
    lens = [n, rng.randint(1, n), rng.randint(1, n)]
    starts = [rng.randint(1, l) for l in lens]
    others = [random_tokens(cfg["vocab"], l, seed + 100 + i) for i, l in enumerate(lens[1:])]
    exact = {}
    tail = min(n - 1, rng.randint(1, 70))
    for kind, dtype in (("sharp", "float32"), ("mild", "float32"), ("mild", "bfloat16")):
        m = load_model(folders[kind], dtype=dtype, max_tokens=2048, device="cuda:0", verbose=False)
        runs = {"whole": run_whole(m, toks), "tail": run_tail_one_by_one(m, toks, tail),
                "pieces": run_in_pieces(m, [toks], [cuts])[0], "batch": run_batched(m, [toks] + others, starts)[0]}
        for what, got in runs.items():
            if kind == "sharp":
                e = row_errors(got, want)
                # sums of float32 through sharp softmaxes and many layers; a fault shows at 1e-2 on more than one row (a close
                # call between experts may fall the other way on one)
                assert e.median() < 1e-4 and int((e > 4e-4).sum()) <= 1, (cfg, what, float(e.median()), float(e.max()))
            elif dtype == "float32":
                exact[what] = got
            else:
                e = row_errors(got, exact[what])
                assert torch.isfinite(got).all() and e.median() < 6e-2, (cfg, what, float(e.median()), float(e.max()))
        m.cache.check()
        assert m.cache.slots.held == 0
        del m
        torch.cuda.empty_cache()
