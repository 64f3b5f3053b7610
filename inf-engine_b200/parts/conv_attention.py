"""Causal grouped-query attention over convolved projections (``ConvAttentionSpec`` states the rule in full).

Per token, with x the mixer's input:

    q, k, v, gate = one product over the row-concatenated weights
    q, k, v       <- short causal convolutions over time, a filter per channel; the last inputs of a sequence are state
    q, k          <- first dimensions of every head turned by position (frequencies may be blended for a long context)
    v             <- kept for later layers of the step, or (1 - lambda) v + lambda v_kept; k and v cached
    o_h           = attention with capped scores and a constant in the softmax's denominator, times sigmoid(gate_h)
    out           = o_proj o

The second to fourth lines are one kernel (``kernels.conv_qkv``), the gate rides in the attention kernels
(``latent.attend_float32``: scores, maxima, weights and sums are float32 whatever the storage type).  The kept values
live in a work buffer of the step: a layer mixes values of the same tokens only, so nothing of them is cached.
"""

from __future__ import annotations

import torch

from .. import kernels
from ..cache.manager import CacheRequirement
from ..weights.loader import ExpectedTensor
from .gated_delta import conv_state_requirement
from .latent import _common_dtype, _rotation, attend_float32
from .linear import Linear, stack_rows
from .registry import build_position, position_class, register_mixer


@register_mixer("conv_attention")
class ConvAttention:
    graph_safe = True          # request bounds, state slots and pages are read on the device

    @staticmethod
    def expected_tensors(spec):
        H, G, d, dv = spec.n_heads, spec.n_kv_heads, spec.head_dim, spec.v_head_dim
        out = {}
        for name, conv, width in ((spec.q_proj, spec.q_conv, H * d), (spec.k_proj, spec.k_conv, G * d), (spec.v_proj, spec.v_conv, G * dv)):
            out[name] = ExpectedTensor((width, spec.hidden))
            if conv is not None:
                out[conv.weight] = ExpectedTensor((width, conv.taps))
        out.update(position_class(spec.position).expected_tensors(spec.position))
        if spec.v_mix is not None:
            out[spec.v_mix] = ExpectedTensor(())
        if spec.head_gate is not None:
            out[spec.head_gate] = ExpectedTensor((H, spec.hidden))
        out[spec.o_proj] = ExpectedTensor((spec.hidden, H * dv))
        return out

    def __init__(self, spec, tensors, rt):
        H, G, d, dv = spec.n_heads, spec.n_kv_heads, spec.head_dim, spec.v_head_dim
        if G <= 0 or H % G:
            raise ValueError(f"{H} query heads are not a multiple of {G} kv heads")
        if not (0 < d <= 256 and 0 < dv <= 256):
            raise ValueError(f"attention kernels take head sizes up to 256, not {d} and {dv}")
        if spec.window is not None and spec.window <= 0:
            raise ValueError("an attention window must be positive")
        convs = [spec.q_conv, spec.k_conv, spec.v_conv]
        if any(c is None for c in convs) and any(c is not None for c in convs):
            raise ValueError("the convolutions of q, k and v come together")
        if convs[0] is not None:
            if len({c.taps for c in convs}) != 1 or not 1 <= convs[0].taps <= kernels.CONV_MAX_TAPS:
                raise ValueError(f"the convolutions of q, k and v share one length of at most {kernels.CONV_MAX_TAPS} taps")
            if any(c.bias is not None for c in convs):
                raise ValueError("the convolutions of q, k and v carry no bias")
        if spec.v_keep and spec.v_mix is not None:
            raise ValueError("a layer keeps its values or mixes kept ones, not both")
        self.spec = spec
        self.rt = rt
        self.position = build_position(spec.position, tensors, rt)
        if _rotation(self.position)[1] > d:
            raise ValueError(f"the rotation turns {_rotation(self.position)[1]} dimensions, a head has {d}")
        ws = [tensors[spec.q_proj], tensors[spec.k_proj], tensors[spec.v_proj]]
        if spec.head_gate is not None:
            ws.append(tensors[spec.head_gate])
        stacked, self.cols = stack_rows(ws, _common_dtype(ws))
        self.proj = Linear(stacked, rt, "conv_attention_proj")
        self.q_width, self.out_width = H * d, H * dv
        self.channels = self.cols[3]               # the convolved columns: queries, keys, values and what lies between
        self.taps = convs[0].taps if convs[0] is not None else 1
        # filters over the same columns, [taps, channels] so that neighbouring channels of a tap lie side by side
        self.conv_weight = None
        if convs[0] is not None:
            filters, _ = stack_rows([tensors[c.weight] for c in convs], torch.float32)
            self.conv_weight = filters.t().contiguous()
        self.v_mode = "keep" if spec.v_keep else ("mix" if spec.v_mix is not None else None)
        self.lam = float(tensors[spec.v_mix].float()) if spec.v_mix is not None else 0.0
        self.sink = torch.full((H,), float(spec.sink), dtype=torch.float32, device=stacked.device) \
            if spec.sink is not None else None
        self.softcap = float(spec.softcap or 0.0)
        self.o = Linear(tensors[spec.o_proj], rt, "o")

    def cache_requirement(self) -> CacheRequirement:
        s = self.spec
        pages = CacheRequirement(kind="kv", n_kv_heads=s.n_kv_heads, head_dim=s.head_dim, window=s.window,
                                 dtype=self.rt.act_dtype, v_head_dim=None if s.v_head_dim == s.head_dim else s.v_head_dim)
        if self.taps == 1:
            return pages
        return CacheRequirement(kind="several", parts=(pages, conv_state_requirement(self.taps, self.channels, self.rt.act_dtype)))

    def forward(self, x: torch.Tensor, ctx, cache) -> torch.Tensor:
        s, rt = self.spec, self.rt
        n = x.shape[0]
        H, G, d, dv = s.n_heads, s.n_kv_heads, s.head_dim, s.v_head_dim
        cols = self.cols
        pages, state = (cache, None) if self.taps == 1 else (cache.parts[0], cache.parts[1].state)
        proj = self.proj(x, rt.ws.take("conv_attn_proj", (n, cols[-1]), rt.act_dtype))
        q = rt.ws.take("conv_attn_q", (n, self.q_width), rt.act_dtype)
        kept = rt.ws.take("kept_values", (n, G * dv), rt.act_dtype) if self.v_mode else None
        kvctx = ctx.kv[pages.group]
        inv_freq, rot_dims, neighbours, mult = _rotation(self.position)
        kpool, vpool = (pages.k, pages.v) if cache.write else (None, None)
        kernels.conv_qkv(proj[:, :self.channels], self.conv_weight, state, q, kpool, vpool, ctx.positions,
                         kvctx.slot_mapping, ctx.q_start, ctx.slots, ctx.n_requests, H, G, d, dv, cols[1], cols[2],
                         ctx.page_size, inv_freq=inv_freq, rot_dims=rot_dims, neighbours=neighbours, mult=mult,
                         v_kept=kept, v_mode=self.v_mode, lam=self.lam, write_state=cache.write, max_q_len=ctx.max_q_len)
        heads = rt.ws.take("conv_attn_out", (n, self.out_width), rt.act_dtype)
        gate = proj[:, cols[3]:cols[3] + H] if s.head_gate is not None else None
        attend_float32(q, heads, pages.k, pages.v, ctx, kvctx, H, G, d, dv, float(s.scale), None, window=s.window,
                       sink=self.sink, softcap=self.softcap, gate=gate)
        return self.o(heads, rt.ws.take("mixer_out", (n, s.hidden), rt.act_dtype))
