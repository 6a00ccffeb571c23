"""Configurations, lively random weights and comparison helpers for the tests of the Fanitar decoder.

The configurations differ from one another and from layer to layer in every size: one to four query heads per kv head, maps of
odd and even size, rotated whole, in part and not at all, values narrower and wider than the two maps together, latents of odd and
even length, windows shorter than a page and of several pages, limits that cut much and little, layers without a
feed-forward, runs of layers passed once to three times.
"""
import json
import os
import sys

import torch

HERE = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, os.path.join(HERE, "plain"))
import fanitar_plain as plain  # noqa: E402

TOL_F32 = 5e-5
TOL_BF16 = 4e-2


def att(heads, kv_heads, dim, vdim, scale, diff, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return "attention", m


def lat(heads, dim, vdim, q_rank, kv_rank, scale, window=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    return "latent_attention", m


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def layer(mixer, mlp=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def config(vocab, width, eps, layers, embed_scale=None, logit_scale=None, loop=None):
    out = {"architecture": "Fanitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if embed_scale is not None:
        out["embedding"] = {"scale": embed_scale}
    if logit_scale is not None:
        out["logit_scale"] = logit_scale
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# odd sizes everywhere; every layer differs from the others; the middle layers passed twice
ODD = config(211, 74, 1e-6, [
    layer(att(3, 1, 10, 7, 0.5, 0.3, rot=(6, 300.0)), dense(33, 0.7)),
    layer(lat(3, 9, 13, 11, 17, 0.4, window=21), dense(28, 2.0)),
    layer(att(6, 2, 5, 19, 0.6, 0.75)),                                                                   # no feed-forward
    layer(lat(5, 4, 6, 23, 5, 0.7), dense(20, 0.3)),
    layer(att(4, 4, 7, 14, 0.4, 0.1, rot=(2, 50.0)), dense(31, 5.0)),
], embed_scale=1.7, logit_scale=0.6, loop=(1, 3, 2))
# sharp attention: large score scales make every softmax pick out single keys
SHARP = config(150, 64, 1e-5, [
    layer(att(4, 2, 16, 32, 2.5, 0.6, rot=(16, 10000.0)), dense(48, 1.5)),
    layer(lat(4, 16, 8, 24, 40, 2.5, window=33), dense(48, 0.9)),
    layer(att(2, 1, 24, 24, 2.0, 0.2, rot=(8, 500.0)), dense(40, 1.1)),
    layer(lat(2, 24, 24, 16, 16, 2.0, window=150)),
], embed_scale=0.8, logit_scale=3.0, loop=(0, 2, 2))
# sizes in multiples of 64: in bfloat16 the products and the attentions run this package's tensor-core kernels
EVEN = config(320, 128, 1e-5, [
    layer(att(4, 2, 64, 128, 0.125, 0.5, rot=(64, 20000.0)), dense(256, 1.3)),
    layer(lat(4, 64, 64, 64, 128, 0.125, window=80), dense(192, 2.0)),
    layer(att(4, 1, 32, 64, 0.18, 0.8, rot=(16, 1000.0)), dense(128, 0.8)),
    layer(att(3, 3, 40, 96, 0.16, 0.3, rot=(40, 10000.0)), dense(320, 3.0)),
    layer(lat(2, 128, 128, 96, 96, 0.09, window=200), dense(64, 1.0)),
], embed_scale=2.0, loop=(0, 3, 2))
CONFIGS = {"odd": (ODD, 8), "sharp": (SHARP, 16), "even": (EVEN, 16)}        # name -> (config, page size)


def lively_tensors(cfg_json, seed, dtype):
    """Random weights under which every mechanism matters: matrices of unit gain, norm weights spread around one, difference
    weights around the layer's constant (seldom close to one, where two maps that agree cancel altogether), sinks between far below and far above the scores, learned rows of the passes as large as
    the stream.  The names and shapes come from the framework's loader; the values are drawn here."""
    from beglin_b200.config import load_config
    from beglin_b200.weights import expected_tensors
    arch, cfg = load_config(dict(cfg_json))
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, role in expected_tensors(arch.build_spec(cfg)).items():
        shape = tuple(role.shape)
        r = lambda *s: torch.randn(*s, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = r(*shape) * 0.5
        elif name == "loop.step":
            t = r(*shape) * 0.5
        elif last in ("norm1", "norm2", "norm1b", "norm2b", "norm"):
            t = 1.0 + 0.2 * r(*shape)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = r(*shape) * (0.3 / shape[0] ** 0.25)
        elif last == "sink":
            t = 1.5 * r(*shape)
        elif last == "b":
            t = r(*shape) * 0.5
        else:
            t = r(*shape) * (1.2 / shape[-1] ** 0.5)
        out[name] = t.to(dtype)
    return out


def write_model(folder, cfg, tensors):
    from beglin_b200.weights import write_safetensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f, indent=1)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return folder


def make_model(root, name, seed=0, dtype=torch.float32, config_json=None):
    """Write a model folder with lively random weights under `root` and return its path."""
    cfg = CONFIGS[name][0] if config_json is None else config_json
    folder = os.path.join(str(root), f"fanitar_{name}_{seed}_{str(dtype).split('.')[-1]}")
    if not os.path.exists(os.path.join(folder, "model.safetensors")):
        write_model(folder, cfg, lively_tensors(cfg, seed, dtype))
    return folder


_CACHE = {}


def plain_logits(folder, ids):
    """float64 logits [T, vocab] of the whole sequence from the plain implementation."""
    if folder not in _CACHE:
        _CACHE[folder] = plain.read_folder(folder, torch.float64)
    key = (folder, tuple(ids))
    if key not in _CACHE:
        cfg, w = _CACHE[folder]
        _CACHE[key] = plain.forward(cfg, w, list(ids))
    return _CACHE[key]


def plain_rounding(folder, ids, dtype=torch.float32):
    """The relative error of the plain implementation with rounded numbers: run in float32 altogether, or (bfloat16) with what an
    engine keeps in that format rounded to it.  So far does rounding alone move this folder's logits: two maps that nearly
    cancel are normed to full size, so single tokens may be ill-conditioned."""
    key = (folder, tuple(ids), dtype)
    if key not in _CACHE:
        cfg, w = plain.read_folder(folder, torch.float32 if dtype == torch.float32 else torch.float64)
        low = plain.exactly if dtype == torch.float32 else (lambda x: x.to(dtype).to(torch.float64))
        _CACHE[key] = rel_err(plain.forward(cfg, w, list(ids), low=low), plain_logits(folder, ids))
    return _CACHE[key]


def rel_err(got, want):
    want = want.to(torch.float64).cpu()
    got = got.to(torch.float64).cpu()
    return float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))


def seeded_ids(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def check_against_plain(got, folder, reqs, tol, rounding=None):
    """got: {(request, position): logits row}; every position of every request against the plain logits.  With `rounding` (a number
    format) a request may be off by three times what rounding to it alone does to the plain implementation, where that is
    more than `tol`."""
    worst, least = 0.0, tol
    for rid, ids in reqs.items():
        tol = least if rounding is None else max(least, 3.0 * plain_rounding(folder, ids, rounding))
        assert tol < 0.5, f"{rid} is all rounding"
        want = plain_logits(folder, ids)
        rows = torch.stack([got[(rid, p)] for p in range(len(ids))])
        assert torch.isfinite(rows).all(), rid
        err = rel_err(rows, want)
        if err > tol:
            per_pos = (rows.double() - want).abs().max(dim=1).values / want.abs().max()
            first = int((per_pos > tol).nonzero()[0])
            raise AssertionError(f"{rid}: relative error {err:.3g} > {tol:g}; first wrong position {first} of {len(ids)}")
        worst = max(worst, err)
    return worst


def poison(engine):
    """NaN in every page: a read of something that was never written, or of what an earlier request left, shows."""
    for g in engine.cache.kv_groups:
        g.device_pool.fill_(float("nan"))
