"""Configurations, lively random weights and comparison helpers for the tests of the Dinatar decoder.

The configurations differ from one another and from layer to layer in every size: one to four query heads per kv head,
values narrower than, as wide as and wider than keys, odd head sizes, windows shorter than a page and of several pages that
keep none, a few or more positions than they hold, recurrences with one to four heads per group, convolutions of one to five
taps, decays through short rows of different lengths with several roots, experts with and without a shared one, one to all of
them per token, layers without a feed-forward, runs of layers passed once to three times.
"""
import json
import os
import sys

import torch

HERE = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, os.path.join(HERE, "plain"))
import dinatar_plain as plain  # noqa: E402

TOL_F32 = 5e-5
TOL_BF16 = 4e-2
# Random configurations in bfloat16: several branches in a row whose results are normed over a row of few features; a fault of
# a kernel shows as an error of the size of the logits themselves.
TOL_BF16_RANDOM = 8e-2
ROUTE_DIMS = 4      # features of the residual that belong to the routers alone in a model with decisive routers


def hgrn2(heads, dim, vdim):
    return "hgrn2", {"heads": heads, "dim": dim, "vdim": vdim}


def gla(heads, dim, vdim, tau, rank):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}


def left(heads, kv_heads, dim, vdim, scale, window=None, keep=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    return m


def right(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def par(l, r):
    return "parallel", {"left": l, "right": r}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        f["shared"] = {"ff": shared}
    return f


def layer(mixer, mlp=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def config(vocab, width, eps, layers, max_positions=768, embed_scale=None, logit_scale=None, loop=None):
    out = {"architecture": "Dinatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_positions": max_positions,
           "layers": layers}
    if embed_scale is not None:
        out["embedding"] = {"scale": embed_scale}
    if logit_scale is not None:
        out["logit_scale"] = logit_scale
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# odd sizes everywhere; every layer differs from the others; the middle layers passed twice
ODD = config(211, 72, 1e-6, [
    layer(gla(3, 10, 7, 4.0, 5), moe(20, 5, 2, shared=28)),
    layer(par(left(6, 2, 9, 13, 0.4, window=17, keep=3), right(3, 8, 11, 1, 3, 2)), dense(33)),
    layer(hgrn2(2, 21, 5), moe(9, 3, 3)),
    layer(par(left(3, 1, 12, 12, 0.3, window=40, keep=50), right(4, 5, 6, 4, 1, 5))),                         # no feed-forward
    layer(hgrn2(1, 6, 31), dense(25)),
], max_positions=333, embed_scale=1.7, logit_scale=0.6, loop=(1, 3, 2))
# sharp attention: large score scales make every softmax pick out single keys
SHARP = config(150, 64, 1e-5, [
    layer(par(left(4, 2, 16, 8, 2.5, window=33, keep=5), right(2, 16, 12, 2, 4, 1)), dense(48)),
    layer(gla(2, 24, 16, 16.0, 9)),
    layer(par(left(2, 1, 24, 24, 2.0, window=150, keep=18), right(4, 8, 16, 2, 2, 4)), moe(16, 4, 1, shared=16)),
], embed_scale=0.8, logit_scale=3.0)
# sizes in multiples of 64: in bfloat16 the products run this package's tensor-core kernels
EVEN = config(320, 128, 1e-5, [
    layer(hgrn2(2, 64, 64), dense(256)),
    layer(par(left(4, 2, 64, 64, 0.125, window=80, keep=4), right(2, 64, 64, 1, 4, 2)), moe(64, 8, 2, shared=128)),
    layer(gla(3, 32, 64, 8.0, 16), moe(128, 4, 3)),
    layer(par(left(2, 2, 128, 128, 0.09, window=200, keep=70), right(4, 32, 32, 2, 4, 1)), dense(192)),
    layer(par(left(8, 1, 32, 64, 0.18), right(2, 64, 16, 2, 3, 4)), moe(64, 2, 1, shared=64)),                  # no window at all
], loop=(0, 2, 2))
CONFIGS = {"odd": (ODD, 8), "sharp": (SHARP, 16), "even": (EVEN, 16)}        # name -> (config, page size)


def lively_tensors(cfg_json, seed, dtype, decisive=False):
    """Random weights under which every mechanism matters: matrices of unit gain, norm weights spread around one, lower bounds
    and decays between forgetting at once and keeping for hundreds of tokens.  The names and shapes come from the framework's
    loader; the values are drawn here.

    `decisive`: for runs in a rounded number format, where a router that reads rounded rows could choose another expert than
    the oracle on a close call.  The last ROUTE_DIMS features of the residual then belong to the routers alone: the embedding
    marks one of them per token, no position vector, shift or sublayer's last matrix writes there, and a router reads nothing
    else, through columns that come in pairs of constant sum: the mean that the layer norm takes off moves all logits alike, and
    their order is the order of one column, whose entries are spaced evenly.  The routers have no bias then."""
    from beglin_b200.config import load_config
    from beglin_b200.weights import expected_tensors
    arch, cfg = load_config(dict(cfg_json))
    spec = arch.build_spec(cfg)
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, role in expected_tensors(spec).items():
        shape = tuple(role.shape)
        r = lambda *s: torch.randn(*s, generator=g)
        u = lambda *s: torch.rand(*s, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = r(*shape) * 0.5
            if decisive:
                t[:, -ROUTE_DIMS:] = 0.0
                t[torch.arange(shape[0]), shape[1] - ROUTE_DIMS + torch.arange(shape[0]) % ROUTE_DIMS] = 3.0
        elif name == "pos":
            t = r(*shape) * 0.4
            if decisive:
                t[:, -ROUTE_DIMS:] = 0.0
        elif name.endswith("router.b"):
            t = torch.zeros(shape) if decisive else r(*shape) * 0.5
        elif last == "router":
            t = r(*shape) * (2.0 / shape[1] ** 0.5)
            if decisive:
                t = torch.zeros(shape)
                for k in range(0, ROUTE_DIMS, 2):
                    col = 1 + torch.randperm(shape[0], generator=g).float()
                    t[:, shape[1] - ROUTE_DIMS + k], t[:, shape[1] - ROUTE_DIMS + k + 1] = 0.5 * col, 0.5 * (shape[0] + 1 - col)
        elif last == "lower":
            t = 0.95 * u(*shape) * (u(*shape) < 0.7).float()       # a third of the channels without a lower bound
        elif name.endswith("mix.f.b"):
            t = 2.0 * r(*shape) + 1.0
        elif name.endswith("a2.b"):
            t = 2.0 * r(*shape) + 2.0
        elif last == "A_log":
            t = 0.7 * r(*shape)
        elif last == "dt_bias":
            t = r(*shape) - 2.0
        elif last == "D":
            t = r(*shape)
        elif name.endswith("norm1.b") or name == "final.norm.b":
            t = 0.3 * r(*shape)
            if decisive and name != "final.norm.b":
                t[-ROUTE_DIMS:] = 0.0
        elif name.endswith("norm1") or name == "final.norm":
            t = 1.0 + 0.2 * r(*shape)
            if decisive and name != "final.norm":
                t[-ROUTE_DIMS:] = 1.0
        elif last in ("norm", "out"):
            t = 1.0 + 0.2 * r(*shape)
        elif last == "b":
            t = r(*shape) * 0.5
        elif last == "conv":
            t = r(*shape) * 0.5
        else:
            t = r(*shape) * (1.2 / shape[-1] ** 0.5)
            if decisive and last in ("o", "down"):
                t[-ROUTE_DIMS:] = 0.0
        out[name] = t.to(dtype)
    return out


def write_model(folder, cfg, tensors):
    """The folder's config.json has no word on the length of a "gla" mixer's short row: the tensor says it."""
    import copy
    from beglin_b200.weights import write_safetensors
    cfg = copy.deepcopy(cfg)
    for l in cfg["layers"]:
        l["mixer"].pop("rank", None)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f, indent=1)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return folder


def make_model(root, name, seed=0, dtype=torch.float32, config_json=None, decisive=None):
    """Write a model folder with lively random weights under `root` and return its path.  A folder stored in bfloat16
    gets decisive routers unless told otherwise."""
    cfg = CONFIGS[name][0] if config_json is None else config_json
    decisive = (dtype != torch.float32) if decisive is None else decisive
    folder = os.path.join(str(root), f"dinatar_{name}_{seed}_{str(dtype).split('.')[-1]}_{int(decisive)}")
    if not os.path.exists(os.path.join(folder, "model.safetensors")):
        write_model(folder, cfg, lively_tensors(cfg, seed, dtype, decisive))
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


def plain_rounding(folder, ids):
    """The relative error of the plain implementation run in float32: how far rounding alone moves this folder's logits (a head's
    result that nearly cancels is normed to full size, so some random weights are ill-conditioned)."""
    key = (folder, "float32")
    if key not in _CACHE:
        _CACHE[key] = plain.read_folder(folder, torch.float32)
    cfg, w = _CACHE[key]
    return rel_err(plain.forward(cfg, w, list(ids)), plain_logits(folder, ids))


def rel_err(got, want):
    want = want.to(torch.float64).cpu()
    got = got.to(torch.float64).cpu()
    return float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))


def seeded_ids(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def check_against_plain(got, folder, reqs, tol):
    """got: {(request, position): logits row}; every position of every request against the plain logits."""
    worst = 0.0
    for rid, ids in reqs.items():
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
    """NaN in every page and state slot: a read of something that was never written, or of what an earlier request
    left, shows."""
    for g in engine.cache.kv_groups:
        g.device_pool.fill_(float("nan"))
    for g in engine.cache.state_groups:
        g.slab.fill_(float("nan"))
