"""Random configurations of the Fanitar decoder: `random_config(case)` is a pure function of the case number and draws every
size, the kinds and the order of the layers, the run that is passed again, windows, rotated parts, limits and the other constants;
each case runs whole and mixed with other requests on a small pool, in float32 and in bfloat16, against the oracle.  The bfloat16
cases draw sizes in multiples of 8 (what the tensor-core products take) and difference weights that stay away from one (at 0.98 a
token whose two maps agree is all rounding in that format)."""
import random

import pytest
import torch

import replay_lib as rl
from fanitar_helpers import (TOL_BF16, TOL_F32, att, check_against_plain, config, dense, lat, layer, make_model,
                             poison, seeded_ids)

pytestmark = pytest.mark.gpu


def random_config(case: int, even: bool = False):
    rng = random.Random(8000 + case)
    unit = 8 if even else 1
    width = rng.choice([64, 128, 192, 200, 320]) if even else rng.randrange(24, 100)

    def mixer():
        if rng.random() < 0.6:
            kv = rng.choice([1, 1, 2, 3])
            heads = kv * rng.choice([1, 1, 2, 3, 4])
            dim = rng.choice([16, 32, 64, 24, 48, 56, 80]) if even else rng.randrange(1, 40)
            vdim = rng.choice([dim, 2 * dim, 2 * dim, 16, 40, 64, 128]) if even else rng.choice([dim, 2 * dim, rng.randrange(1, 60)])
            dims = rng.choice([0, dim, dim // 2]) // (2 * unit) * (2 * unit) if even else rng.randrange(0, dim + 1) // 2 * 2
            rot = None if rng.random() < 0.2 else (dims, rng.choice([50.0, 10000.0, 500000.0]))
            return att(heads, kv, dim, vdim, rng.uniform(0.3, 2.0) / dim ** 0.5, rng.uniform(0.05, 0.6 if even else 0.9), rot)
        heads = rng.randrange(1, 7)
        dim = rng.choice([16, 32, 64, 128, 40]) if even else rng.randrange(1, 40)
        vdim = rng.choice([dim, dim, 16, 32, 64]) if even else rng.choice([dim, rng.randrange(1, 40)])
        rank = lambda: rng.choice([32, 64, 96, 128, 40, 72]) if even else rng.randrange(1, 60)
        return lat(heads, dim, vdim, rank(), rank(), rng.uniform(0.3, 2.0) / dim ** 0.5,
                   rng.choice([None, 1, 2, rng.randrange(3, 20), rng.randrange(20, 200)]))

    n = rng.randrange(1, 5)
    layers = [layer(mixer(), None if rng.random() < 0.2 else dense(unit * rng.randrange(1, 40), rng.choice([0.3, 1.0, 2.5, 7.0])))
              for _ in range(n)]
    start = rng.randrange(0, n)
    loop = rng.choice([None, (start, rng.randrange(start + 1, n + 1), rng.randrange(1, 4))])
    cfg = config(rng.randrange(30, 300), width, rng.choice([1e-6, 1e-5, 1e-3]), layers, embed_scale=rng.choice([None, 0.5, 2.5]),
                 logit_scale=rng.choice([None, 0.3, 4.0]), loop=loop)
    return cfg, rng.choice([4, 8, 16, 32, 64])


@pytest.mark.parametrize("case", list(range(14)) + [15, 34])      # 15 and 34: heads, or a latent, of a single feature
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_random_configuration(model_root, case, dtype):
    cfg, page = random_config(case, even=(dtype == "bfloat16"))
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    folder = make_model(model_root, f"random{case}", seed=case, dtype=stored, config_json=cfg)
    reqs = {f"r{i}": seeded_ids(n, cfg["vocab"], 7 * case + i) for i, n in enumerate([61, 18, 130, 40, 77])}
    mixed_steps, peak = rl.mixed(reqs, seed=case)
    from beglin_b200 import Engine
    results = {}
    tol = TOL_F32 if dtype == "float32" else TOL_BF16
    for way, (steps, tokens) in {"whole": (rl.whole(reqs), 192), "mixed": (mixed_steps, peak)}.items():
        eng = Engine.from_folder(folder, dtype=dtype, max_tokens=max(tokens, page), page_size=page, max_requests=4, kv_split=64 if case % 2 else 256)
        poison(eng)
        results[way] = rl.run_in_process(eng, steps)
        eng.cache.check()
        check_against_plain(results[way], folder, reqs, tol, stored)
    if dtype == "float32":
        for key, row in results["whole"].items():
            assert torch.equal(results["mixed"][key], row), key
