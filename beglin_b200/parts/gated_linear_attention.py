"""Linear attention with a decay per key channel (HGRN2's forget gate, gated linear attention's rooted sigmoid).

One product of the mixer's input gives, side by side, the rows for q, for the forget gate or the keys, for v, for the gate on
the result and for the short row that the decays are made from, as far as the spec has them.  Per head, for each token in turn
    S <- diag(a) S + k v^T;    o = S^T q
with, for `write` "forget", a = l + (1 - l) sigmoid(f + b) and k = 1 - a, and for `write` "key", k a product of its own and
a = sigmoid(W2 r + b)^power for the short row r = W1 h.  Each head's o is RMS-normed by itself (and multiplied by silu of the
gate), and the joined heads go through the output product.

The state S is per-request state of fixed size (one slot of the cache manager's slab, float32, zero when the request starts):
a step continues each request from its slot, however the request's tokens are cut into steps and whatever else the step holds.
Behind the products everything is float in both number formats, up to the heads' normed rows.

Requests that bring `LONG_FROM` rows or more walk them in chunks: the chunks' own sums and outputs are computed side by side
and only a pass over the chunks' states is serial.  Fewer rows, and single tokens, are walked one by one.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..csrc import ops
from .cache_need import FixedStateNeed, FixedStateView
from .context import BuildContext
from .linear import Linear
from .registry import register_mixer
from .spec import GatedLinearAttentionSpec, TensorRole
from .stream import NormedInput, ResidualStream


@register_mixer("gated_linear_attention")
class GatedLinearAttention:
    LONG_FROM = 16             # rows of a request in a step from which its tokens run in chunks

    @staticmethod
    def expected_tensors(spec: GatedLinearAttentionSpec) -> List[TensorRole]:
        qd, vd, d = spec.n_heads * spec.dim, spec.n_heads * spec.vdim, spec.hidden
        roles = [TensorRole("q_proj.weight", (qd, d), True, True)]
        if spec.write == "forget":
            roles += [TensorRole("f_proj.weight", (qd, d), True, True), TensorRole("f_proj.bias", (qd,), role="bias"),
                      TensorRole("lower", (qd,))]
        else:
            roles += [TensorRole("k_proj.weight", (qd, d), True, True), TensorRole("decay_in.weight", (spec.decay_rank, d), True, True),
                      TensorRole("decay_out.weight", (qd, spec.decay_rank), True, True),
                      TensorRole("decay_out.bias", (qd,), role="bias")]
        roles.append(TensorRole("v_proj.weight", (vd, d), True, True))
        if spec.gated:
            roles.append(TensorRole("g_proj.weight", (vd, d), True, True))
        return roles + [TensorRole("norm.weight", (spec.vdim,), role="scale"), TensorRole("o_proj.weight", (d, vd), True, True)]

    @staticmethod
    def cache_need(spec: GatedLinearAttentionSpec) -> FixedStateNeed:
        return FixedStateNeed((spec.n_heads * spec.dim * spec.vdim,), "float32")

    def __init__(self, spec: GatedLinearAttentionSpec, tensors: Dict[str, torch.Tensor], ctx: BuildContext):
        if spec.write not in ("forget", "key"):
            raise ValueError(f"unknown way of writing '{spec.write}' (forget, key)")
        if spec.write == "key" and (spec.decay_rank < 1 or not spec.decay_power > 0.0):
            raise ValueError("the decays want a positive rank and a positive power")
        self.spec, self.ctx = spec, ctx
        self.qd, self.vd = spec.n_heads * spec.dim, spec.n_heads * spec.vdim
        names = ["q_proj", "f_proj" if spec.write == "forget" else "k_proj", "v_proj"] + (["g_proj"] if spec.gated else [])
        rows = [tensors[n + ".weight"] for n in names]
        self.g_col = 2 * self.qd + self.vd if spec.gated else -1
        self.r_col = sum(w.shape[0] for w in rows)
        if spec.write == "key":
            rows.append(tensors["decay_in.weight"])
        pad = -sum(w.shape[0] for w in rows) % 8       # rows of zeros keep the product's rows 16 bytes apart
        if pad:
            rows.append(torch.zeros((pad, spec.hidden), dtype=rows[0].dtype, device=rows[0].device))
        self.in_proj = Linear(torch.cat(rows, dim=0), None, ctx, label="proj_qkv")
        self.o_proj = Linear(tensors["o_proj.weight"], None, ctx, label="proj_o")
        f32 = lambda t: t.to(device=ctx.device, dtype=torch.float32).contiguous()
        self.norm_w = f32(tensors["norm.weight"])
        if spec.write == "forget":
            self.bias, self.lower, self.decay_w = f32(tensors["f_proj.bias"]), f32(tensors["lower"]), None
        else:
            self.bias, self.lower, self.decay_w = f32(tensors["decay_out.bias"]), None, f32(tensors["decay_out.weight"])
        self.chunk = ops.gla_chunk(spec.dim, spec.vdim) if ctx.device.type == "cuda" else 0

    takes_stream = True        # forward takes a NormedInput and may add its result to the stream itself

    def forward(self, h, batch, cache: FixedStateView, stream: Optional[ResidualStream] = None) -> Optional[torch.Tensor]:
        """h: the normed rows, or a NormedInput.  With `stream` the result is added to it (or left owed to it) and None
        is returned; without, the addend is returned."""
        if isinstance(h, NormedInput):
            h = h.tensor()
        s = self.spec
        proj = self.in_proj.full_f32(h)                                 # [T, q | f or k | v (| gate) (| short row)]
        if self.chunk and not batch.decode_only and hasattr(batch, "long_blocks"):
            reqs, n_req, chunks, n_chunks, longs, n_long = batch.long_blocks(self.chunk, self.LONG_FROM)
        else:
            reqs, n_req = batch.query_blocks(1 << 30)                   # one (request, first row, rows) per request
            chunks, n_chunks, longs, n_long = None, 0, None, 0
        out = torch.empty((batch.n_rows, self.vd), dtype=self.ctx.compute_dtype, device=h.device)
        ops.gated_linear_attention(proj, 0, self.qd, 2 * self.qd, self.bias, self.norm_w, s.eps, cache.state, cache.slots, reqs, n_req,
                                   out, s.n_heads, s.dim, s.vdim, lower=self.lower, decay_matrix=self.decay_w, r_col=self.r_col,
                                   power=s.decay_power, q_silu=s.query_silu, q_scale=s.query_scale, g_col=self.g_col,
                                   chunks=chunks, n_chunks=n_chunks, longs=longs, n_long=n_long)
        if stream is None:
            return self.o_proj.partial(out)
        self.o_proj.into(out, stream)
        return None
