"""Random configurations of the Dinatar decoder: `random_config(case)` is a pure function of the case number and draws every
size, the kinds and the order of the layers, the run that is passed again, windows and kept positions, the experts' numbers and
the constants; each case runs whole and mixed with other requests on a small pool, in float32 and in bfloat16, against the
oracle.  The bfloat16 cases draw sizes in multiples of 8 (what the tensor-core products take) and routers that no rounding can
turn (see `lively_tensors`)."""
import random

import pytest
import torch

import replay_lib as rl
from dinatar_helpers import (TOL_BF16_RANDOM, TOL_F32, check_against_plain, config, dense, gla, hgrn2, layer, left, make_model, moe, par,
                             plain_rounding, poison, rel_err, right, seeded_ids)

pytestmark = pytest.mark.gpu


def random_config(case: int, even: bool = False):
    rng = random.Random(7000 + case)
    unit = 8 if even else 1
    width = rng.choice([64, 128, 192, 200, 320]) if even else rng.randrange(24, 100)

    def mixer():
        kind = rng.choice(["hgrn2", "gla", "parallel"])
        if kind != "parallel":
            heads = rng.randrange(1, 5)
            dim = rng.choice([16, 32, 48, 64, 96, 128]) if even else rng.randrange(1, 50)
            vdim = rng.choice([16, 32, 40, 64, 128]) if even else rng.randrange(1, 50)
            return hgrn2(heads, dim, vdim) if kind == "hgrn2" else gla(heads, dim, vdim, rng.choice([1.0, 3.5, 16.0]), rng.randrange(1, 40))
        kv = rng.choice([1, 1, 2, 3])
        heads = kv * rng.choice([1, 1, 2, 3, 4])
        dim = rng.choice([32, 64, 128, 48, 80, 96]) if even else rng.randrange(1, 40)
        vdim = rng.choice([dim, dim, 16, 32, 64, 40]) if even else rng.choice([dim, rng.randrange(1, 40)])
        window = rng.choice([None, 1, 2, rng.randrange(3, 20), rng.randrange(20, 200)])
        keep = rng.choice([None, 0, 1, rng.randrange(2, 12), rng.randrange(12, 150)])
        groups = rng.randrange(1, 4)
        rh = groups * rng.randrange(1, 4)
        p = unit * rng.randrange(1, 6) if even else rng.randrange(1, 20)
        parts = rng.choice([g for g in range(1, 7) if (rh * p) % g == 0])
        return par(left(heads, kv, dim, vdim, rng.uniform(0.3, 2.0) / dim ** 0.5, window, keep),
                   right(rh, p, rng.choice([8, 16, 48, 64]) if even else rng.randrange(1, 40), groups, rng.randrange(1, 6), parts))

    def feed_forward():
        r = rng.random()
        if r < 0.2:
            return None
        if r < 0.55:
            return dense(unit * rng.randrange(1, 40))
        experts = rng.randrange(1, 9)
        return moe(unit * rng.randrange(1, 20), experts, rng.randrange(1, min(experts, 4) + 1), rng.choice([None, unit * rng.randrange(1, 20)]))

    n = rng.randrange(1, 5)
    layers = [layer(mixer(), feed_forward()) for _ in range(n)]
    start = rng.randrange(0, n)
    loop = rng.choice([None, (start, rng.randrange(start + 1, n + 1), rng.randrange(1, 4))])
    cfg = config(rng.randrange(30, 300), width, rng.choice([1e-6, 1e-5, 1e-3]), layers, max_positions=rng.choice([130, 200, 1000]),
                 embed_scale=rng.choice([None, 0.5, 2.5]), logit_scale=rng.choice([None, 0.3, 4.0]), loop=loop)
    return cfg, rng.choice([4, 8, 16, 32, 64])


@pytest.mark.parametrize("case", range(14))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_random_configuration(model_root, case, dtype):
    cfg, page = random_config(case, even=(dtype == "bfloat16"))
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    folder = make_model(model_root, f"random{case}", seed=case, dtype=stored, config_json=cfg)
    reqs = {f"r{i}": seeded_ids(n, cfg["vocab"], 7 * case + i) for i, n in enumerate([61, 18, 130, 40, 77])}
    mixed_steps, peak = rl.mixed(reqs, seed=case)
    from beglin_b200 import Engine
    results = {}
    tol = max(TOL_F32, 4.0 * max(plain_rounding(folder, ids) for ids in reqs.values())) if dtype == "float32" else TOL_BF16_RANDOM
    assert tol < 1e-3 or dtype == "bfloat16"
    for way, (steps, tokens) in {"whole": (rl.whole(reqs), 192), "mixed": (mixed_steps, peak)}.items():
        eng = Engine.from_folder(folder, dtype=dtype, max_tokens=max(tokens, page), page_size=page, max_requests=4, kv_split=64)
        poison(eng)
        results[way] = rl.run_in_process(eng, steps)
        eng.cache.check()
        check_against_plain(results[way], folder, reqs, tol)
    if dtype == "float32":
        for key, row in results["whole"].items():
            assert rel_err(results["mixed"][key], row) < 2 * tol, key      # (two roundings of their own)
