"""Causal grouped-query attention whose values are the projected keys before their rotation (``TiedAttentionSpec``): there is
no value projection.

Per token, with x the mixer's input:

    q, k = one product over the row-concatenated weights, biases added
    v    = k
    q, k <- first dimensions of every head turned by position
    o    = attention over the keys of the query's own chunk of positions, or over all earlier ones
    out  = o_proj o

Biases, rotation and the cache write of keys and values are one kernel (``kernels.head_prepare`` with ``tied``), scores,
maxima, weights and sums are float32 whatever the storage type (``latent.attend_float32``).  A layer that rotates nothing
keeps one pool: its values are its key rows.
"""

from __future__ import annotations

import torch

from .. import kernels
from ..cache.manager import CacheRequirement
from ..weights.loader import ExpectedTensor
from .latent import _common_dtype, _rotation, attend_float32
from .linear import Linear, stack_rows
from .registry import build_position, position_class, register_mixer


@register_mixer("tied_attention")
class TiedAttention:
    graph_safe = True          # positions, slots and pages are read on the device

    @staticmethod
    def expected_tensors(spec):
        H, G, d = spec.n_heads, spec.n_kv_heads, spec.head_dim
        out = {}
        for name, bias, width in ((spec.q_proj, spec.q_bias, H * d), (spec.k_proj, spec.k_bias, G * d)):
            out[name] = ExpectedTensor((width, spec.hidden))
            if bias is not None:
                out[bias] = ExpectedTensor((width,))
        out.update(position_class(spec.position).expected_tensors(spec.position))
        out[spec.o_proj] = ExpectedTensor((spec.hidden, H * d))
        return out

    def __init__(self, spec, tensors, rt):
        H, G, d = spec.n_heads, spec.n_kv_heads, spec.head_dim
        if G <= 0 or H % G:
            raise ValueError(f"{H} query heads are not a multiple of {G} kv heads")
        if not 0 < d <= 256:
            raise ValueError(f"attention kernels take head sizes up to 256, not {d}")
        self.spec = spec
        self.rt = rt
        self.position = build_position(spec.position, tensors, rt)
        if _rotation(self.position)[1] > d:
            raise ValueError(f"the rotation turns {_rotation(self.position)[1]} dimensions, a head has {d}")
        ws = [tensors[spec.q_proj], tensors[spec.k_proj]]
        stacked, self.cols = stack_rows(ws, _common_dtype(ws))
        self.proj = Linear(stacked, rt, "tied_proj")
        biases = [tensors[n] for n in (spec.q_bias, spec.k_bias) if n is not None]
        pick = lambda n: tensors[n].to(_common_dtype(biases)).contiguous() if n is not None else None
        self.q_bias, self.k_bias = pick(spec.q_bias), pick(spec.k_bias)
        self.rotates = _rotation(self.position)[0] is not None
        self.o = Linear(tensors[spec.o_proj], rt, "o")

    def cache_requirement(self) -> CacheRequirement:
        s = self.spec
        return CacheRequirement(kind="kv", n_kv_heads=s.n_kv_heads, head_dim=s.head_dim, dtype=self.rt.act_dtype,
                                chunk=s.chunk, values_in_keys=not self.rotates)

    def forward(self, x: torch.Tensor, ctx, cache) -> torch.Tensor:
        s, rt = self.spec, self.rt
        n = x.shape[0]
        H, G, d = s.n_heads, s.n_kv_heads, s.head_dim
        proj = self.proj(x, rt.ws.take("tied_proj", (n, self.cols[-1]), rt.act_dtype))
        q, k = proj[:, :H * d], proj[:, self.cols[1]:self.cols[1] + G * d]
        kvctx = ctx.kv[cache.group]
        inv_freq, rot_dims, neighbours, mult = _rotation(self.position)
        kpool, vpool = (cache.k, cache.v) if cache.write else (None, None)
        kernels.head_prepare(q, H, d, k, G, d, ctx.positions, kvctx.slot_mapping, kpool, ctx.page_size,
                             inv_freq=inv_freq, rot_dims=rot_dims, neighbours=neighbours, mult=mult, q_bias=self.q_bias,
                             k_bias=self.k_bias, tied=self.rotates, vpool=vpool if self.rotates else None)
        heads = rt.ws.take("tied_out", (n, H * d), rt.act_dtype)
        attend_float32(q, heads, cache.k, cache.v, ctx, kvctx, H, G, d, d, float(s.scale), s.chunk)
        return self.o(heads, rt.ws.take("mixer_out", (n, s.hidden), rt.act_dtype))
