"""Plain, slow implementation of the Fanitar decoder, used only as the oracle of the tests.

Whole sequences, no cache, one function per mechanism, float64 tensor arithmetic on the CPU.  It shares no code with the
`beglin_b200` package: the model folder is read with the `json` module and the `safetensors` library, and attention is
computed query by query over explicit lists of visible keys, so that a fault of the engine's loader, cache, batching or
kernels cannot be mirrored here.

The design in this file's notation.  The stream starts as s E[token].  A layer norms a sublayer's input AND its result:
x <- x + N1b(M(N1(x))), then x <- x + N2b(F(N2(x))) (a layer may lack F); N is the RMS norm with a weight of its own at
every place.  A run of layers may be passed several times: in front of pass t the stream gets the embedded rows once more
(t > 0) and a learned row P[t].  The logits are c W N(x).

Mixers: "attention" is grouped-query attention whose heads come as pairs of maps over the same values, the second map's
result taken off the first's times one learned number of the layer, the difference normed to unit mean square;
"latent_attention" makes queries, keys and values from short normed rows, has no positions, a sliding window, one learned
score per head in the softmax's denominator that carries no value, and a sigmoid gate per feature.

Feed-forward: W_down of a gated activation whose two branches are cut off at a limit.
"""
from __future__ import annotations

import json
import math
import os
from typing import Callable, Dict, List, Optional, Sequence

import torch

SLOPE = 1.702          # of the sigmoid inside the gated activation


def exactly(x: torch.Tensor) -> torch.Tensor:
    """The default of `low`: nothing is rounded.  (`forward` with another `low` passes through it what an engine in a rounded number
    format keeps in that format, which tells how far rounding alone moves the logits.)"""
    return x



def read_folder(folder: str, dtype: torch.dtype = torch.float64):
    from safetensors import safe_open

    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    weights: Dict[str, torch.Tensor] = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            weights[name] = f.get_tensor(name).to(dtype)
    return cfg, weights


# ----------------------------------------------------------------------------- small functions
def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_unit(x, eps) * w


def turn_halves(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, ..., n] with the token's position as first index: feature i < dims/2 turns together with feature i + dims/2 by
    position * base^(-2i/dims); features from dims on pass."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        f = base ** (-2.0 * i / dims)
        c = torch.tensor([math.cos(t * f) for t in range(x.shape[0])], dtype=x.dtype).view(-1, *[1] * (x.dim() - 2))
        s = torch.tensor([math.sin(t * f) for t in range(x.shape[0])], dtype=x.dtype).view(-1, *[1] * (x.dim() - 2))
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


# ----------------------------------------------------------------------------- attention, query by query
def visible(t: int, size: Optional[int]) -> List[int]:
    """The keys that query t sees: itself and, with a window, the size - 1 before it."""
    return [j for j in range(t + 1) if size is None or t - j < size]


def plain_softmax_weights(s: torch.Tensor, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """exp(s_j) / (sum_j exp(s_j) + exp(sink)) over the first index, the last term only where given."""
    top = s.amax(0) if sink is None else torch.maximum(s.amax(0), sink)
    e = torch.exp(s - top)
    z = e.sum(0) + (0.0 if sink is None else torch.exp(sink - top))
    return e / z


def two_maps(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float):
    """q [T, H, 2, n], k [T, G, 2, n], v [T, G, m] -> (a1, a2), each [T, H, m]: the attentions of the first and the second
    map, over the same values; query head h reads kv head h // (H / G)."""
    T, H = q.shape[:2]
    G = k.shape[1]
    reads = [h // (H // G) for h in range(H)]
    k, v = k[:, reads], v[:, reads]                                     # what each query head reads
    out = [torch.zeros((T, H, v.shape[2]), dtype=q.dtype) for _ in range(2)]
    for t in range(T):
        keys = visible(t, None)
        for c in range(2):
            p = plain_softmax_weights((k[keys, :, c] * q[t, :, c]).sum(-1) * scale)             # [keys, H]
            out[c][t] = (p[:, :, None] * v[keys]).sum(0)
    return out


def difference_weight(w: Dict[str, torch.Tensor], diff: float) -> torch.Tensor:
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def differential_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, low: Callable = exactly) -> torch.Tensor:
    T = h.shape[0]
    H, G, n, nv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, 2, n)
    k = (h @ w["k"].T + w["k.b"]).view(T, G, 2, n)
    v = (h @ w["v"].T + w["v.b"]).view(T, G, nv)
    rot = m.get("rot")
    if rot is not None and rot["dims"] > 0:
        q, k = turn_halves(q, rot["base"], rot["dims"]), turn_halves(k, rot["base"], rot["dims"])
    a1, a2 = two_maps(low(q), low(k), low(v), m["scale"])
    o = rms_unit(a1 - difference_weight(w, m["diff"]) * a2, eps) * (1.0 - m["diff"])
    return low(o).reshape(T, H * nv) @ w["o"].T


def latent_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, low: Callable = exactly) -> torch.Tensor:
    T = h.shape[0]
    H, n, nv = m["heads"], m["dim"], m["vdim"]
    q = low(low(rms_norm(h @ w["dq"].T, w["dq.norm"], eps)) @ w["uq"].T).view(T, H, n)
    c = low(rms_norm(h @ w["dkv"].T, w["dkv.norm"], eps))
    k, v = low(c @ w["uk"].T).view(T, H, n), low(c @ w["uv"].T).view(T, H, nv)
    size = (m.get("mask") or {}).get("size")
    o = torch.zeros((T, H, nv), dtype=h.dtype)
    for t in range(T):
        keys = visible(t, size)
        p = plain_softmax_weights((k[keys] * q[t]).sum(-1) * m["scale"], w["sink"])             # [keys, H]
        o[t] = (p[:, :, None] * v[keys]).sum(0)
    return low(o.reshape(T, H * nv) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ----------------------------------------------------------------------------- feed-forward
def cut_gate(g: torch.Tensor, u: torch.Tensor, limit: float) -> torch.Tensor:
    """The gate is cut above, the other branch on both sides."""
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(SLOPE * g) * (u + 1.0)


def feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], f: dict, low: Callable = exactly) -> torch.Tensor:
    if f["kind"] != "dense":
        raise ValueError(f["kind"])
    return low(cut_gate(low(h @ w["gate"].T), low(h @ w["up"].T), f["limit"])) @ w["down"].T


# ----------------------------------------------------------------------------- the model
def sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def mixer_of(kind: str, h, w, m, eps, low=exactly):
    if kind == "attention":
        return differential_mixer(h, w, m, eps, low)
    if kind == "latent_attention":
        return latent_mixer(h, w, m, eps, low)
    raise ValueError(kind)


def run_order(n_layers: int, loop: Optional[dict]):
    """[(layer, the number of the pass that begins in front of it, or None)]."""
    if loop is None:
        return [(i, None) for i in range(n_layers)]
    lo, hi = loop["start"], loop["stop"]
    out = [(i, None) for i in range(lo)]
    for t in range(loop["times"]):
        out += [(i, t if i == lo else None) for i in range(lo, hi)]
    return out + [(i, None) for i in range(hi, n_layers)]


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: Sequence[int], tap: Optional[Callable] = None,
            low: Callable = exactly) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence from position 0.  `tap(run, rows)` gets the stream behind every layer run."""
    eps = cfg["norm"]["eps"]
    scale = (cfg.get("embedding") or {}).get("scale", 1.0)
    e = weights["embed"][list(tokens)] * scale
    x = e.clone()
    for ri, (li, begins) in enumerate(run_order(len(cfg["layers"]), cfg.get("loop"))):
        layer, p = cfg["layers"][li], f"l{li}."
        if begins is not None:
            if begins > 0:
                x = x + e
            x = x + weights["loop.step"][begins]
        y = mixer_of(layer["type"], low(rms_norm(x, weights[p + "norm1"], eps)), sub(weights, p + "mix."), layer["mixer"], eps, low)
        x = x + rms_norm(low(y), weights[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(low(rms_norm(x, weights[p + "norm2"], eps)), sub(weights, p + "mlp."), layer["mlp"], low)
            x = x + rms_norm(low(y), weights[p + "norm2b"], eps)
        if tap is not None:
            tap(ri, x)
    x = low(rms_norm(x, weights["final.norm"], eps))
    return (x @ weights["head"].T) * cfg.get("logit_scale", 1.0)
