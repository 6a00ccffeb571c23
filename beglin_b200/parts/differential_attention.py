"""Differential attention over the paged cache: every head is a pair of attention maps over the same values.

Per head the two maps' results a1 and a2 are joined to o = a1 - lambda a2, which is divided by its root mean square and
multiplied by 1 - diff; lambda is one number of the layer, made when the model is built from four learned vectors.

To the kernels this is grouped-query attention in which a page of a kv head holds the keys of both maps side by side, one row
of 2 x dim features per position, and ONE value: a query head counts as two, each of which meets its own half of the key row.
So a page's keys and values are read once for both maps and all query heads of the kv head.  Where the two queries of a head
are told apart depends on the kernel: the CUDA-core and the tcgen05 kernels multiply only the map's half of a key row; the
decoding kernel, which is bound by the bytes of the cache, takes queries with zeros in the other map's half.  The difference
and its norm are float: they are the last step of the tcgen05 kernel, and elsewhere of the kernel that merges the ranges of keys.

A step: one product for q, k and v (with their biases), one kernel for the rotation and the append, attention, and the output
product.  In bfloat16 a map's features are stored 32 or 64 wide, zeros behind its own, so that the rows have the 64 or 128
features that the tensor-core kernels take.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import numpy as np
import torch

from ..csrc import ops
from .cache_need import PagedKVNeed, PagedKVView
from .context import BuildContext
from .linear import Linear
from .registry import register_mixer
from .rope import shared_position
from .spec import DifferentialAttentionSpec, TensorRole
from .stream import ResidualStream

MAPS = 2


@register_mixer("differential_attention")
class DifferentialAttention:
    @staticmethod
    def expected_tensors(spec: DifferentialAttentionSpec) -> List[TensorRole]:
        sizes = (("q", spec.n_heads * MAPS * spec.dim), ("k", spec.n_kv_heads * MAPS * spec.dim), ("v", spec.n_kv_heads * spec.vdim))
        roles = [TensorRole(f"{x}_proj.weight", (n, spec.hidden), True, True) for x, n in sizes]
        if spec.qkv_bias:
            roles += [TensorRole(f"{x}_proj.bias", (n,), role="bias") for x, n in sizes]
        roles += [TensorRole(v, (spec.dim,)) for v in ("lq1", "lk1", "lq2", "lk2")]
        return roles + [TensorRole("o_proj.weight", (spec.hidden, spec.n_heads * spec.vdim), True, True)]

    cache_need_takes_context = True        # cache_need(spec, ctx): what a page holds depends on the compute type

    @staticmethod
    def stored(spec: DifferentialAttentionSpec, ctx: Optional[BuildContext]) -> Tuple[int, int]:
        """(features of a stored map, of a stored value): as they are, or, in bfloat16, as wide as the tensor-core kernels take
        them where that does not more than double the cache."""
        if ctx is not None and ctx.compute_dtype == torch.bfloat16 and ctx.cache_dtype == torch.bfloat16 and ctx.attention != "generic":
            for wide in (64, 128):
                if MAPS * spec.dim <= wide and spec.vdim <= wide:
                    if wide <= MAPS * spec.dim + spec.vdim:
                        return wide // MAPS, wide
                    break
        return spec.dim, spec.vdim

    @staticmethod
    def cache_need(spec: DifferentialAttentionSpec, ctx: Optional[BuildContext] = None) -> PagedKVNeed:
        kw, vw = DifferentialAttention.stored(spec, ctx)
        return PagedKVNeed(spec.n_kv_heads, MAPS * kw, spec.window, None if vw == MAPS * kw else vw)

    def __init__(self, spec: DifferentialAttentionSpec, tensors: Dict[str, torch.Tensor], ctx: BuildContext):
        if spec.n_heads % spec.n_kv_heads:
            raise ValueError(f"{spec.n_heads} query heads are not a multiple of {spec.n_kv_heads} kv heads")
        self.spec, self.ctx = spec, ctx
        self.nh, self.nkv, self.dim, self.vd = spec.n_heads, spec.n_kv_heads, spec.dim, spec.vdim
        w = torch.cat([tensors[f"{x}_proj.weight"] for x in "qkv"], dim=0)
        b = torch.cat([tensors[f"{x}_proj.bias"].float() for x in "qkv"], dim=0) if spec.qkv_bias else None
        pad = -w.shape[0] % 8                          # rows of zeros keep the product's rows 16 bytes apart
        if pad:
            w = torch.cat([w, torch.zeros((pad, w.shape[1]), dtype=w.dtype, device=w.device)], dim=0)
            b = None if b is None else torch.cat([b, torch.zeros(pad, dtype=b.dtype, device=b.device)])
        self.qkv = Linear(w, b, ctx, label="proj_qkv")
        self.o_proj = Linear(tensors["o_proj.weight"], None, ctx, label="proj_o")
        self.position = shared_position(spec.position, ctx)
        if self.position.rotary_dim > spec.dim:
            raise ValueError(f"{self.position.rotary_dim} rotated features of a map of {spec.dim}")
        self.scale = float(np.float32(spec.scale))
        v64 = lambda n: tensors[n].to(device="cpu", dtype=torch.float64)
        lam = torch.exp((v64("lq1") * v64("lk1")).sum()) - torch.exp((v64("lq2") * v64("lk2")).sum()) + float(spec.diff)
        self.lam, self.out_scale = float(np.float32(float(lam))), float(np.float32(1.0 - float(spec.diff)))
        self.kw, self.vw = self.stored(spec, ctx)
        self.window = int(spec.window) if spec.window else 0
        self.plans = {d: ops.difference_plan(self.nh // self.nkv, self.kw, self.vw, ctx.cache_dtype, d, ctx.attention, ctx.page_size)
                      for d in (False, True)}

    takes_stream = True        # forward takes a NormedInput and may add its result to the stream itself

    def forward(self, h, batch, cache: PagedKVView, stream: Optional[ResidualStream] = None) -> Optional[torch.Tensor]:
        """h: the normed rows, or a NormedInput.  With `stream` the result is added to it (or left owed to it) and None
        is returned; without, the addend is returned."""
        ctx, T = self.ctx, batch.n_rows
        qkv = self.qkv.of(h)
        kernel, bq, tile = self.plans[bool(getattr(batch, "decode_only", False))]
        padded = kernel == "mma_keys"                  # queries with zeros where the other map's keys lie
        q = torch.empty((T, MAPS * self.nh * self.kw * (MAPS if padded else 1)), dtype=ctx.compute_dtype, device=qkv.device)
        ops.qk_norm_rope_append(qkv, q, T, MAPS * self.nh, self.nkv, self.dim, self.vd, self.position.rotary_dim,
                                self.position.interleaved, None, None, 0.0, self.position.table(batch), batch.positions,
                                batch.row_req, cache.block_table, cache.pool, cache.page_size, ctx.status,
                                maps=MAPS, stored=(self.kw, self.vw), padded=padded)
        qblk, n_qblk = batch.query_blocks(bq)
        if qblk is None and kernel != "mma_keys":
            batch.implicit_blocks = False              # this kernel wants the list
            qblk, n_qblk = batch.query_blocks(bq)
        out = torch.empty((T, self.nh * self.vd), dtype=ctx.compute_dtype, device=q.device)
        ops.difference_attention(q, cache.pool, cache.block_table, batch.positions, qblk, n_qblk, batch.max_position, T, self.nh,
                                 self.nkv, self.kw, self.vw, self.vd, self.window, ctx.kv_split, tile, bq, self.scale, self.lam,
                                 self.out_scale, self.spec.eps, out, ctx.status, kernel)
        if stream is None:
            return self.o_proj.partial(out)
        self.o_proj.into(out, stream)
        return None
