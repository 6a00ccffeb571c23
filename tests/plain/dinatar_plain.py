"""Plain, slow implementation of the Dinatar decoder, used only as the oracle of the tests.

Whole sequences, no cache, one function per mechanism, float64 tensor arithmetic on the CPU.  It shares no code with the
`beglin_b200` package: the model folder is read with the `json` module and the `safetensors` library, attention is
computed query by query over explicit lists of visible keys, the recurrences token by token and the experts token by
token, so that a fault of the engine's loader, cache, batching or kernels cannot be mirrored here.

The design in this file's notation.  The stream starts as s E[token] + P[position].  A layer forms ONE normed copy
h = LN(x) = (x - mean) / sqrt(mean((x - mean)^2) + eps) g + b and adds two results to the stream, x <- x + M(h) + F(h)
(a layer may lack F).  A run of layers may be passed several times.  The logits are c E LN(x).

Mixers: "hgrn2" and "gla" are linear attention with a decay per key channel, S <- diag(a) S + k v^T read out as S^T q,
every head's result normed by itself; in the first a = l + (1 - l) sigmoid(.) and k = 1 - a, in the second a is a
sigmoid's tau-th root and the joined heads meet a SiLU gate.  "parallel" is grouped-query attention with a falling line
per head on the scores and a sliding window that never loses the first few tokens, beside a Mamba-2 recurrence; each
branch's result is normed over the width and the two are averaged.

Feed-forward: W_down relu(W_up h)^2, or gated experts with a biased router whose weights are a softmax over the chosen
logits, beside an expert for every token.
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, List, Optional, Sequence

import torch


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


def layer_norm(x: torch.Tensor, g: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * g + b


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


# ----------------------------------------------------------------------------- linear attention with a decay per key channel
def decayed_readout(q: torch.Tensor, k: torch.Tensor, a: torch.Tensor, v: torch.Tensor,
                    state: Optional[torch.Tensor] = None):
    """q, k, a [T, H, n], v [T, H, m] -> (o [T, H, m], the state behind the last token).  Per head, token by token:
    S <- diag(a_t) S + k_t v_t^T;  o_t = S^T q_t."""
    T, H, n = q.shape
    s = torch.zeros((H, n, v.shape[2]), dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        s = a[t][:, :, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (s * q[t][:, :, None]).sum(1)
    return out, s


def forget_gate(z: torch.Tensor, lower: torch.Tensor) -> torch.Tensor:
    return lower + (1.0 - lower) * torch.sigmoid(z)


def rooted_decay(z: torch.Tensor, tau: float) -> torch.Tensor:
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def hgrn2_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, n, nv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).view(T, H, n)
    a = forget_gate(h @ w["f"].T + w["f.b"], w["lower"]).view(T, H, n)
    v = (h @ w["v"].T).view(T, H, nv)
    o, _ = decayed_readout(q, 1.0 - a, a, v)
    return (rms_unit(o, eps) * w["norm"]).reshape(T, H * nv) @ w["o"].T


def gla_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, n, nv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, n) * n ** -0.5
    k = (h @ w["k"].T).view(T, H, n)
    v = (h @ w["v"].T).view(T, H, nv)
    a = rooted_decay((h @ w["a1"].T) @ w["a2"].T + w["a2.b"], m["tau"]).view(T, H, n)
    o, _ = decayed_readout(q, k, a, v)
    o = (rms_unit(o, eps) * w["norm"]).reshape(T, H * nv)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


# ----------------------------------------------------------------------------- attention, query by query
def visible(t: int, size: Optional[int], keep_first: int) -> List[int]:
    """The keys that query t sees: itself and the size - 1 before it, and the sequence's first `keep_first`."""
    return [j for j in range(t + 1) if size is None or t - j < size or j < keep_first]


def falling_slope(h: int, H: int) -> float:
    return 2.0 ** (-8.0 * (h + 1) / H)


def sloped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, see: Callable[[int], List[int]],
                     slopes: Optional[Sequence[float]]) -> torch.Tensor:
    """q [T, H, n], k [T, G, n], v [T, G, nv] -> [T, H, nv]; query head h reads kv head h // (H / G); the score of key j
    falls by slopes[h] for every position it lies back."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for t in range(T):
        keys = see(t)
        back = torch.tensor([float(t - j) for j in keys], dtype=q.dtype)
        for h in range(H):
            g = h // (H // G)
            s = (k[keys, g] @ q[t, h]) * scale
            if slopes is not None:
                s = s - slopes[h] * back
            out[t, h] = torch.softmax(s, dim=-1) @ v[keys, g]
    return out


def attention_branch(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, n, nv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, n)
    k = (h @ w["k"].T + w["k.b"]).view(T, G, n)
    v = (h @ w["v"].T + w["v.b"]).view(T, G, nv)
    mask = m.get("mask") or {}
    o = sloped_attention(q, k, v, m["scale"], lambda t: visible(t, mask.get("size"), mask.get("keep_first", 0)),
                         [falling_slope(hh, H) for hh in range(H)])
    return o.reshape(T, H * nv) @ w["o"].T


# ----------------------------------------------------------------------------- Mamba-2
def causal_taps(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, K] (the last column meets the current token), zeros before the start."""
    T, C = x.shape
    K = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        acc = bias.clone()
        for j in range(K):
            src = t - (K - 1 - j)
            if src >= 0:
                acc = acc + taps[:, j] * x[src]
        out[t] = acc
    return out


def mamba2_branch(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(causal_taps(xbc, w["conv"], w["conv.b"]))
    x = xbc[:, :inner].view(T, H, P)
    B = xbc[:, inner:inner + G * N].view(T, G, N)
    C = xbc[:, inner + G * N:].view(T, G, N)
    dt = torch.nn.functional.softplus(dt + w["dt_bias"])
    s = torch.zeros((H, N, P), dtype=h.dtype)
    y = torch.zeros((T, H, P), dtype=h.dtype)
    for t in range(T):
        for hh in range(H):
            g = hh // (H // G)
            s[hh] = torch.exp(-torch.exp(w["A_log"][hh]) * dt[t, hh]) * s[hh] + dt[t, hh] * torch.outer(B[t, g], x[t, hh])
            y[t, hh] = s[hh].T @ C[t, g] + w["D"][hh] * x[t, hh]
    y = y.reshape(T, inner) * silu(z)
    parts = m["norm_groups"]
    y = rms_unit(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w["norm"]
    return y @ w["o"].T


def parallel_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    left = attention_branch(h, sub(w, "left."), m["left"])
    right = mamba2_branch(h, sub(w, "right."), m["right"], eps)
    return 0.5 * (rms_unit(left, eps) * w["left.out"] + rms_unit(right, eps) * w["right.out"])


# ----------------------------------------------------------------------------- feed-forward
def gated_expert(h: torch.Tensor, w: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    return (silu(h @ w[name + ".gate"].T) * (h @ w[name + ".up"].T)) @ w[name + ".down"].T


def routed_feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], f: dict) -> torch.Tensor:
    E, top = f["router"]["experts"], f["router"]["top"]
    z = h @ w["router"].T + w["router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(E), key=lambda e: (-float(z[t, e]), e))[:top]
        share = torch.softmax(z[t, order], dim=-1)
        for c, e in zip(share, order):
            out[t] = out[t] + c * gated_expert(h[t], w, f"e{e}")
    if f.get("shared") is not None:
        out = out + gated_expert(h, w, "shared")
    return out


def feed_forward(h: torch.Tensor, w: Dict[str, torch.Tensor], f: dict) -> torch.Tensor:
    if f["kind"] == "dense":
        return relu_squared(h @ w["up"].T) @ w["down"].T
    if f["kind"] == "moe":
        return routed_feed_forward(h, w, f)
    raise ValueError(f["kind"])


# ----------------------------------------------------------------------------- the model
def sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def mixer_of(kind: str, h, w, m, eps):
    if kind == "hgrn2":
        return hgrn2_mixer(h, w, m, eps)
    if kind == "gla":
        return gla_mixer(h, w, m, eps)
    if kind == "parallel":
        return parallel_mixer(h, w, m, eps)
    raise ValueError(kind)


def run_order(n_layers: int, loop: Optional[dict]) -> List[int]:
    if loop is None:
        return list(range(n_layers))
    lo, hi = loop["start"], loop["stop"]
    return list(range(lo)) + list(range(lo, hi)) * loop["times"] + list(range(hi, n_layers))


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: Sequence[int], tap: Optional[Callable] = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence from position 0.  `tap(run, rows)` gets the stream behind every layer run."""
    eps = cfg["norm"]["eps"]
    scale = (cfg.get("embedding") or {}).get("scale", 1.0)
    x = weights["embed"][list(tokens)] * scale + weights["pos"][:len(tokens)]
    for ri, li in enumerate(run_order(len(cfg["layers"]), cfg.get("loop"))):
        layer, p = cfg["layers"][li], f"l{li}."
        h = layer_norm(x, weights[p + "norm1"], weights[p + "norm1.b"], eps)
        y = mixer_of(layer["type"], h, sub(weights, p + "mix."), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, sub(weights, p + "mlp."), layer["mlp"])
        x = x + y
        if tap is not None:
            tap(ri, x)
    x = layer_norm(x, weights["final.norm"], weights["final.norm.b"], eps)
    return (x @ weights["embed"].T) * cfg.get("logit_scale", 1.0)
