"""A mixture of feed-forward experts (gated, or without a gate), chosen and run on the device: a sigmoid or softmax router with groups, or
(``score`` "softmax_top") the largest logits plus a bias, weighted by the softmax over the chosen logits alone.

Per token, with x the part's input (``RoutedExpertsSpec`` states the rule in full):

    s = sigmoid(router x)                      float32 products and sums
    choice = s + correction                    for the choice only; groups of experts, the best groups kept
    chosen = the ``top`` largest choice scores among the kept groups
    weight = s[chosen] / (sum of them + eps) * route_scale
    out = sum weight_e * down_e(silu(gate_e x) * up_e x)  +  sigmoid(shared_gate x) * shared(x)

The router's product also carries the shared expert's gate, if there is one (one more row).  Nothing waits for the device: the
(token, choice) pairs are sorted by expert in one small kernel, and two grouped products walk the sorted pairs in
tiles that never span two experts (``csrc/routed.cu``), so the part may sit inside a captured decode step.  Prompt
portions in bfloat16 that give the experts enough rows run both products on the tcgen05 tensor cores, over rows gathered
into sorted order; a few tokens stream the chosen experts' weights.  A pair's result does not depend on where it lands in
the sorted order, nor (beyond the rounding of another kernel's order of sums) on what else the step holds.
"""

from __future__ import annotations

import torch

from .. import kernels
from ..weights.loader import ExpectedTensor
from .feedforward import MLP_ACTIVATIONS
from .linear import Linear
from .registry import build_feedforward, feedforward_class, register_feedforward


@register_feedforward("routed_experts")
class RoutedExperts:
    graph_safe = True

    @staticmethod
    def expected_tensors(spec):
        out = {}
        for e in range(spec.n_experts):
            p = f"{spec.expert_prefix}{e}."
            if spec.gated:
                out[p + "gate"] = ExpectedTensor((spec.intermediate, spec.hidden))
            out[p + "up"] = ExpectedTensor((spec.intermediate, spec.hidden))
            out[p + "down"] = ExpectedTensor((spec.hidden, spec.intermediate))
        out[spec.router] = ExpectedTensor((spec.n_experts, spec.hidden))
        if spec.correction is not None:
            out[spec.correction] = ExpectedTensor((spec.n_experts,))
        if spec.router_bias is not None:
            out[spec.router_bias] = ExpectedTensor((spec.n_experts,))
        if spec.shared is not None:
            out.update(feedforward_class(spec.shared).expected_tensors(spec.shared))
            if spec.shared_gate is not None:
                out[spec.shared_gate] = ExpectedTensor((1, spec.hidden))
        return out

    def __init__(self, spec, tensors, rt):
        E = spec.n_experts
        if E % spec.n_groups or not 0 < spec.keep_groups <= spec.n_groups:
            raise ValueError(f"{E} experts in {spec.n_groups} groups of which {spec.keep_groups} are kept: not possible")
        if not 0 < spec.top <= spec.keep_groups * (E // spec.n_groups):
            raise ValueError(f"{spec.top} experts cannot be chosen from {spec.keep_groups} groups of {E // spec.n_groups}")
        if spec.score not in kernels.ROUTE_SCORES:
            raise ValueError(f"router score {spec.score!r} is not built (known: {', '.join(kernels.ROUTE_SCORES)})")
        if spec.score == "softmax_top" and (spec.n_groups != 1 or spec.correction is not None):
            raise ValueError("a router whose weights are the softmax over the chosen logits has no groups and no correction")
        if spec.score != "softmax_top" and spec.router_bias is not None:
            raise ValueError("a bias of the router's logits belongs to the softmax over the chosen logits")
        if spec.group_score not in kernels.GROUP_SCORES:
            raise ValueError(f"group score {spec.group_score!r} is not built (known: {', '.join(kernels.GROUP_SCORES)})")
        known = sorted(kernels.GLU_KINDS) if spec.gated else list(MLP_ACTIVATIONS)
        if spec.activation not in known:
            raise ValueError(f"activation {spec.activation!r} is not built (known: {known})")
        if spec.shared_gate is not None and spec.shared is None:
            raise ValueError("a shared expert's gate without a shared expert")
        # the activation in the first product's epilogue
        self.act = kernels.glu_constants(spec.activation, spec.act_alpha, spec.act_limit, spec.up_offset) if spec.gated else None
        self.epi = "silu_mul" if spec.gated else spec.activation
        self.spec = spec
        self.rt = rt
        names = [f"{spec.expert_prefix}{e}." for e in range(E)]
        every = [tensors[p + k] for p in names for k in (("gate", "up", "down") if spec.gated else ("up", "down"))]
        dtype = torch.float32 if any(t.dtype is torch.float32 for t in every) else every[0].dtype
        # [experts, 2 * intermediate, hidden] with rows alternating gate_j, up_j: a thread of the product's epilogue
        # then holds both halves of a pair; [experts, hidden, intermediate] for the way back
        # (without a gate: [experts, intermediate, hidden])
        if spec.gated:
            self.first = torch.stack([torch.stack([tensors[p + "gate"].to(dtype), tensors[p + "up"].to(dtype)], dim=1)
                                      .reshape(2 * spec.intermediate, spec.hidden) for p in names]).contiguous()
        else:
            self.first = torch.stack([tensors[p + "up"].to(dtype) for p in names]).contiguous()
        self.down = torch.stack([tensors[p + "down"].to(dtype) for p in names]).contiguous()
        self.gated_shared = spec.shared_gate is not None
        rows = [tensors[spec.router]] + ([tensors[spec.shared_gate].reshape(1, spec.hidden)] if self.gated_shared else [])
        rdtype = torch.float32 if any(t.dtype is torch.float32 for t in rows) else rows[0].dtype
        self.router = torch.cat([t.to(rdtype) for t in rows], dim=0).contiguous()
        self.correction = tensors[spec.correction].contiguous() if spec.correction is not None else None
        if spec.router_bias is not None:
            self.correction = tensors[spec.router_bias].contiguous()      # the route kernel adds it to the logits
        self.shared = build_feedforward(spec.shared, tensors, rt) if spec.shared is not None else None

    TCGEN05_MIN_ROWS = 32      # rows an expert gets on average from which tiles of 128 rows on tcgen05 pay

    def _on_tcgen05(self, x: torch.Tensor, n_pairs: int) -> bool:
        s = self.spec
        return (self.rt.act_dtype is torch.bfloat16 and x.dtype is torch.bfloat16 and self.first.dtype is torch.bfloat16
                and self.down.dtype is torch.bfloat16 and n_pairs >= self.TCGEN05_MIN_ROWS * s.n_experts and x.shape[0] >= 128
                and s.hidden % 64 == 0 and s.intermediate % 64 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0)

    def _run_experts(self, x: torch.Tensor):
        """(the chosen experts' results [n * top, hidden] float32, their weights [n, top], the shared expert's gate)."""
        s, rt, ws = self.spec, self.rt, self.rt.ws
        n, E, top = x.shape[0], s.n_experts, s.top
        n_pairs = n * top
        logits = ws.take("moe_logits", (n, self.router.shape[0]), torch.float32)
        # float32 products and sums whatever the activation type; few outputs: a warp per (token, expert)
        (kernels.gemm_rowdot if self.router.shape[0] <= 128 else kernels.gemm_simt)(x, self.router, logits)
        ids = ws.take("moe_ids", (n, top), torch.int32)
        weights = ws.take("moe_weights", (n, top), torch.float32)
        gate = ws.take("moe_gate", (n,), torch.float32) if self.shared is not None else None     # (1 without a gate tensor)
        kernels.moe_route(logits, self.correction, ids, weights, gate, E, top, s.n_groups, s.keep_groups, s.route_scale,
                          s.weight_eps, gate_col=E if self.gated_shared else -1, score=s.score, group_score=s.group_score)
        sorted_pairs = ws.take("moe_sorted", (n_pairs,), torch.int32)
        hidden = ws.take("moe_hidden", (n_pairs, s.intermediate), rt.act_dtype)       # in sorted order
        y = ws.take("moe_pairs_out", (n_pairs, s.hidden), torch.float32)               # in the pairs' own order
        if self._on_tcgen05(x, n_pairs):
            rows = kernels.gemm_tcgen05_tile_rows()
            tiles = ws.take("moe_tiles", (kernels.moe_max_tiles(n_pairs, E, rows), 4), torch.int32)
            kernels.moe_sort(ids, E, sorted_pairs, tiles, rows)
            xs = ws.take("moe_rows", (n_pairs, s.hidden), torch.bfloat16)
            kernels.moe_gather(x, xs, sorted_pairs, top)
            kernels.gemm_tcgen05_grouped(xs, self.first, hidden, tiles, None, self.epi, act=self.act)
            kernels.gemm_tcgen05_grouped(hidden, self.down, y, tiles, sorted_pairs, "f32")
            return y, weights, gate
        tiles = ws.take("moe_tiles", (kernels.moe_max_tiles(n_pairs, E), 4), torch.int32)
        kernels.moe_sort(ids, E, sorted_pairs, tiles)
        kernels.moe_gemm(x, self.first, hidden, sorted_pairs, tiles, top, gather=True, scatter=False, epi=self.epi,
                         act=self.act)
        kernels.moe_gemm(hidden, self.down, y, sorted_pairs, tiles, top, gather=False, scatter=True)
        return y, weights, gate

    @property
    def forward_unsummed(self):
        """``(y, weights, more)`` for a caller that forms ``sum_r weights[n, r] * y[n * top + r]`` plus the rows of ``more``
        (the shared expert's, if there is one) itself, or None where there is more to the result than that sum."""
        return self._unsummed if not self.gated_shared else None

    def _unsummed(self, x: torch.Tensor, ctx):
        y, weights, _ = self._run_experts(x)
        return y, weights, (self.shared.forward(x, ctx),) if self.shared is not None else ()

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        y, weights, gate = self._run_experts(x)
        shared = self.shared.forward(x, ctx) if self.shared is not None else None
        out = self.rt.ws.take("moe_out", (x.shape[0], self.spec.hidden), torch.float32)
        kernels.moe_combine(y, weights, gate, shared, out)
        return out
