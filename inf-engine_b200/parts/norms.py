"""RMSNorm: ``x / sqrt(mean(x^2) + eps) * gain`` (engine/layers.py:11-25), with
float32 statistics whatever the activation dtype, fused with the residual sum
that precedes it in a pre-norm block (engine/llama_block.py:53-62).  With
``unit_offset`` the stored tensor lies around zero and the gain is one plus it
(formed once, in float32); with ``scalar`` the stored tensor is a single number that multiplies every coordinate.
``accumulate`` is the norm of a block that norms its
sublayers' OUTPUTS: the normed rows are added into the residual.
``GroupedRMSNorm`` norms each of several equal consecutive parts of the row by itself, and takes a summand that carries
a multiplier per coordinate or is a mixture of experts not summed up yet (``ScaledDelta``) in the same kernel.
``TanhNorm`` (dynamic tanh) has no statistics: ``tanh(alpha x) * gain + bias``, coordinate by coordinate, with such a summand
taken in the same way.
LayerNorm: ``(x - mean) / sqrt(variance + eps) * weight + bias`` with the variance
the mean of the squared deviations, the same way."""

from __future__ import annotations

import torch

from .. import kernels
from ..weights.loader import ExpectedTensor
from .registry import register_norm


class ScaledDelta:
    """A summand of the residual stream that is not added yet: ``mult * scale * (y + sum of extras)`` with ``scale``
    float32 [d] (None: 1), or, with ``weights`` float32 [n, top], ``sum_r weights[n, r] * y[n * top + r]`` in the place of
    y.  ``extras``: up to two results of sublayers that read the same input, of one type."""

    __slots__ = ("y", "scale", "weights", "mult", "extras")

    def __init__(self, y: torch.Tensor, scale: torch.Tensor | None = None, weights: torch.Tensor | None = None,
                 mult: float = 1.0, extras: tuple = ()):
        self.y, self.scale, self.weights, self.mult, self.extras = y, scale, weights, mult, extras


def add_pending(residual: torch.Tensor, pending) -> None:
    """residual += pending, a tensor or a ``ScaledDelta``."""
    if isinstance(pending, ScaledDelta):
        kernels.stream_norm(residual, pending.y, pending.scale, pending.weights, None, 1, 0.0, None, mult=pending.mult,
                            extras=pending.extras)
    else:
        kernels.residual_add(residual, pending)


def plain_delta(residual: torch.Tensor, delta):
    """``delta`` as the norms that take a tensor or nothing want it: a ``ScaledDelta`` is added here and now."""
    if isinstance(delta, ScaledDelta):
        add_pending(residual, delta)
        return None
    return delta


@register_norm("rmsnorm")
class RMSNorm:
    @staticmethod
    def expected_tensors(spec):
        return {spec.weight: ExpectedTensor(() if getattr(spec, "scalar", False) else (spec.size,), init="gain")}

    def __init__(self, spec, tensors, rt):
        self.spec = spec
        self.rt = rt
        self.gain = tensors[spec.weight]
        if getattr(spec, "scalar", False):
            # one number for every coordinate: spread out once, so that the kernels and the products that apply a norm
            # in their prologue see the vector they expect
            self.gain = self.gain.reshape(1).expand(spec.size).contiguous()
        if getattr(spec, "unit_offset", False):
            self.gain = (1.0 + self.gain.float()).contiguous()
        self.eps = float(spec.eps)
        self.size = spec.size

    def accumulate(self, residual: torch.Tensor, y: torch.Tensor, next_in: torch.Tensor | None = None) -> None:
        """residual += norm(y); ``next_in`` (activation type, optional) takes the new residual rows."""
        kernels.outnorm_accumulate(residual, y, self.gain, self.eps, next_in)

    def accumulate_then_norm(self, residual: torch.Tensor, y: torch.Tensor, next_norm, out_name: str = "normed"):
        """residual += norm(y), and in the same kernel the rows that ``next_norm`` (an RMS norm of this size) makes of
        the new residual; None when the two do not go together (the caller then runs them one after the other)."""
        if not isinstance(next_norm, RMSNorm) or next_norm.size != self.size or next_norm.gain.dtype != self.gain.dtype:
            return None
        out = self.rt.ws.take(out_name, tuple(residual.shape), self.rt.act_dtype)
        kernels.outnorm_accumulate_norm(residual, y, self.gain, self.eps, next_norm.gain, next_norm.eps, out)
        return out

    def fusable_rms(self):
        """(gain, eps) for kernels that apply this norm inside a matrix product's prologue."""
        return self.gain, self.eps

    def add_norm(self, residual: torch.Tensor, delta: torch.Tensor | None, out_name: str = "normed") -> torch.Tensor:
        out = self.rt.ws.take(out_name, tuple(residual.shape), self.rt.act_dtype)
        kernels.rmsnorm(residual, plain_delta(residual, delta), self.gain, out, self.eps)
        return out

    def gather_norm(self, residual: torch.Tensor, delta: torch.Tensor | None, row_index: torch.Tensor,
                    n_rows: int, out_name: str = "normed_rows") -> torch.Tensor:
        out = self.rt.ws.take(out_name, (n_rows, self.size), self.rt.act_dtype)
        kernels.rmsnorm(residual, plain_delta(residual, delta), self.gain, out, self.eps, row_index=row_index)
        return out


@register_norm("grouped_rmsnorm")
class GroupedRMSNorm:
    """RMS norm of each of ``groups`` equal consecutive parts of the row by itself; the whole times the gain (and a
    constant, formed into the gain once)."""

    @staticmethod
    def expected_tensors(spec):
        return {spec.weight: ExpectedTensor((spec.size,), init="gain")}

    def __init__(self, spec, tensors, rt):
        if spec.groups <= 0 or spec.size % spec.groups:
            raise ValueError(f"a row of {spec.size} does not split into {spec.groups} equal parts")
        self.spec = spec
        self.rt = rt
        self.gain = tensors[spec.weight].contiguous()
        if spec.out_scale != 1.0:
            self.gain = (self.gain.float() * spec.out_scale).contiguous()
        self.eps = float(spec.eps)
        self.size = spec.size
        self.groups = int(spec.groups)

    def _norm(self, residual, delta, out, row_index=None):
        d = delta if isinstance(delta, ScaledDelta) else ScaledDelta(delta)
        kernels.stream_norm(residual, d.y, d.scale, d.weights, self.gain, self.groups, self.eps, out, row_index,
                            mult=d.mult, extras=d.extras)
        return out

    def add_norm(self, residual: torch.Tensor, delta, out_name: str = "normed") -> torch.Tensor:
        return self._norm(residual, delta, self.rt.ws.take(out_name, tuple(residual.shape), self.rt.act_dtype))

    def gather_norm(self, residual: torch.Tensor, delta, row_index: torch.Tensor, n_rows: int,
                    out_name: str = "normed_rows") -> torch.Tensor:
        return self._norm(residual, delta, self.rt.ws.take(out_name, (n_rows, self.size), self.rt.act_dtype), row_index)


@register_norm("tanh_norm")
class TanhNorm:
    """Dynamic tanh: ``tanh(alpha x) * gain + bias``, coordinate by coordinate, alpha one number of the model's."""

    @staticmethod
    def expected_tensors(spec):
        return {spec.weight: ExpectedTensor((spec.size,), init="gain"), spec.bias: ExpectedTensor((spec.size,)),
                spec.alpha: ExpectedTensor((), init="gain")}

    def __init__(self, spec, tensors, rt):
        self.spec = spec
        self.rt = rt
        self.gain, self.bias = tensors[spec.weight].contiguous(), tensors[spec.bias].contiguous()
        if self.gain.dtype != self.bias.dtype:
            self.gain, self.bias = self.gain.float(), self.bias.float()
        self.tanh = (float(tensors[spec.alpha].float()), self.bias)
        self.size = spec.size

    def _norm(self, residual, delta, out, row_index=None):
        d = delta if isinstance(delta, ScaledDelta) else ScaledDelta(delta)
        kernels.stream_norm(residual, d.y, d.scale, d.weights, self.gain, 1, 0.0, out, row_index, mult=d.mult,
                            extras=d.extras, tanh=self.tanh)
        return out

    def add_norm(self, residual: torch.Tensor, delta, out_name: str = "normed") -> torch.Tensor:
        return self._norm(residual, delta, self.rt.ws.take(out_name, tuple(residual.shape), self.rt.act_dtype))

    def gather_norm(self, residual: torch.Tensor, delta, row_index: torch.Tensor, n_rows: int,
                    out_name: str = "normed_rows") -> torch.Tensor:
        return self._norm(residual, delta, self.rt.ws.take(out_name, (n_rows, self.size), self.rt.act_dtype), row_index)


@register_norm("layernorm")
class LayerNorm:
    @staticmethod
    def expected_tensors(spec):
        out = {spec.weight: ExpectedTensor((spec.size,), init="gain")}
        if spec.bias is not None:
            out[spec.bias] = ExpectedTensor((spec.size,))
        return out

    def __init__(self, spec, tensors, rt):
        self.spec = spec
        self.rt = rt
        self.weight = tensors[spec.weight]
        self.bias = tensors[spec.bias].to(self.weight.dtype) if spec.bias is not None else None
        self.eps = float(spec.eps)
        self.size = spec.size

    def add_norm(self, residual: torch.Tensor, delta: torch.Tensor | None, out_name: str = "normed") -> torch.Tensor:
        out = self.rt.ws.take(out_name, tuple(residual.shape), self.rt.act_dtype)
        kernels.layernorm(residual, plain_delta(residual, delta), self.weight, self.bias, out, self.eps)
        return out

    def gather_norm(self, residual: torch.Tensor, delta: torch.Tensor | None, row_index: torch.Tensor,
                    n_rows: int, out_name: str = "normed_rows") -> torch.Tensor:
        out = self.rt.ws.take(out_name, (n_rows, self.size), self.rt.act_dtype)
        kernels.layernorm(residual, plain_delta(residual, delta), self.weight, self.bias, out, self.eps, row_index=row_index)
        return out
