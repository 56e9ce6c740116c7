"""Gudarax configurations drawn at random (every size and constant that config.json gives, layer by layer, in any order of
the three mixers and the three feed-forwards) in cuttings drawn at random too (whole, a tail one by one, pieces, unequal
batches): in 32-bit against the plain implementation on weights that make attention sharp, and in bfloat16 against the
32-bit engine on a milder scale of the same configuration."""
import os
import random

import pytest
import torch

from cima_b200.engine import load_model
from gudarax_cases import attention, config, delta, dense, latent, moe, row_errors, write_folder
from gudarax_plain import plain_forward, read_folder
from helpers import random_tokens, run_batched, run_in_pieces, run_tail_one_by_one, run_whole

pytestmark = pytest.mark.gpu

SEEDS = list(range(int(os.environ.get("CIMA_RANDOM_CONFIGS", "8"))))


def draw_mlp(rng: random.Random):
    r = rng.random()
    if r < 0.15:
        return None
    if r < 0.45:
        return dense(rng.choice([8, 20, 33, 64, 96, 130]))
    experts = rng.choice([1, 2, 3, 5, 8, 13, 40])
    return moe(experts, rng.randint(1, min(experts, 5)), rng.choice([7, 8, 16, 24, 40, 64]))


def draw_config(rng: random.Random) -> dict:
    width = rng.choice([16, 24, 25, 32, 48, 64, 80, 100, 128, 192, 320])            # some are no multiple of 8
    shared = (rng.choice([1, 2, 3]), rng.choice([8, 16, 20, 24, 32, 48, 64, 80, 128]))    # key heads and value size of the mixing layers
    layers = []
    for _ in range(rng.randint(1, 6)):
        r = rng.random()
        if r < 0.45:
            mix = rng.random() < 0.6
            kv, vdim = shared if mix else (rng.choice([1, 2, 3]), rng.choice([8, 16, 20, 32, 64, 100, 128]))
            dim = rng.choice([8, 16, 20, 32, 48, 64, 80, 96, 128])
            layers.append(attention(kv * rng.choice([1, 2, 4]), kv, dim, vdim, rng.choice([0.5, 1.0, 4.0]) * dim ** -0.5,
                                    rng.choice([0, 1, 3, 40, 63, 64, 65, 100, 128, 200, 1000]), mix, draw_mlp(rng)))
        elif r < 0.72:
            dim = rng.choice([8, 16, 24, 40, 64, 80])
            layers.append(latent(rng.randint(1, 5), dim, rng.choice([8, 12, 32, 64, 65]), rng.choice([8, 16, 17, 40, 64, 80, 128, 136]),
                                 rng.choice([4, 9, 16, 48, 100]), rng.choice([0.5, 1.0, 3.0]) * dim ** -0.5, draw_mlp(rng)))
        else:
            kv = rng.choice([1, 2, 3])
            layers.append(delta(kv * rng.choice([1, 2, 3]), kv, rng.choice([1, 8, 16, 24, 32, 48, 64, 100, 136]), rng.choice([8, 20, 32, 64, 65, 96]),
                                rng.choice([1, 2, 3, 4, 7]), draw_mlp(rng)))
    return config(rng.choice([129, 333, 512, 1001]), width, rng.choice([600, 777]), rng.choice([1e-6, 1e-5, 3e-4]), rng.choice([0.5, 1.0, 4.0]),
                  rng.choice([1, 4, 7, 16, 40]), layers)


@pytest.mark.parametrize("seed", SEEDS)
def test_random_configuration(seed, tmp_path):
    rng = random.Random(13000 + seed)
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
    tail = min(n - 1, rng.randint(1, 130))
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
