"""Norm parts.  ``rms``: ``weight * x * rsqrt(mean(x^2) + eps)`` with the statistics in float32
(miniserve/model/layers.py:30-34), fused with the residual add that precedes it.  ``one_plus``: the stored weight
lies around zero and stands for ``1 + weight`` (added once, in float32, when the weight is loaded).  ``identity``: no norm
at all, for blocks whose sublayers read the residual stream itself: what is pending is added and the stream is handed on in
the compute type.  ``layer``: layer norm with weight and bias, ``weight * (x - mean) / sqrt(mean((x - mean)^2) + eps) + bias``;
two of them that read the same stream run as one kernel (``add_and_norm_both``).  ``dynamic_tanh``: no statistics at all, entry by
entry ``weight * tanh(alpha * x) + bias`` with one ``alpha`` per norm."""

from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from .base import ChannelScaled, ParamSpec, Part, PostNormed, StreamVector, register_norm


@register_norm("rms")
class RMSNorm(Part):
    def __init__(self, *, name: str, size: int, eps: float, prefix: str = "", one_plus: bool = False) -> None:
        self.name, self.size, self.eps = prefix + name, size, float(eps)
        self.one_plus = bool(one_plus)
        self.weight: Optional[torch.Tensor] = None

    def param_specs(self) -> list[ParamSpec]:
        return [ParamSpec(self.name, (self.size,), "vector")]

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self.name]
        if self.one_plus:
            self.weight = (self.weight.float() + 1.0).contiguous()

    def add_and_norm(self, residual: torch.Tensor, delta, out: torch.Tensor,
                     rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``residual += delta`` (float32, in place; skipped when ``delta`` is None), ``out = norm(residual)``.
        ``delta`` may be a pair of tensors (a block whose mixer and feed-forward read the same input hands on both
        outputs): the stream then receives their float32 sum.

        With ``rows`` only those rows are normalised into ``out [len(rows), size]`` and the
        residual stays as it is.
        """
        if isinstance(delta, PostNormed):
            # the output of the sublayer before passes its own norm on the way into the stream: one kernel for both
            kernels.postnorm_add_rmsnorm(residual, delta.x, delta.weight, delta.eps, self.weight, self.eps, out, rows,
                                         post_scale=delta.scale)
            return out
        if isinstance(delta, ChannelScaled):
            # the output of the sublayer before is multiplied channel by channel (in float32) on its way into the stream
            kernels.postnorm_add_rmsnorm(residual, delta.x, delta.weight, 0.0, self.weight, self.eps, out, rows, post_norm=False)
            return out
        if isinstance(delta, StreamVector):
            kernels.add_bias(residual, delta.vector)
            delta = None
        second = None
        if isinstance(delta, tuple):
            delta, second = delta
        kernels.add_rmsnorm(residual, delta, self.weight, self.eps, out, rows, second)
        return out

    def fold(self) -> tuple[torch.Tensor, float]:
        """(weight, eps): all that the products around this norm need to carry it out between them."""
        return self.weight, self.eps

    def norm(self, x: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        """Norm over the last dim of ``x`` (any leading shape) without a residual."""
        kernels.rmsnorm(x, self.weight, self.eps, out)
        return out


@register_norm("identity")
class IdentityNorm(Part):
    """The place of a norm in a block whose sublayers read the stream as it is (designs that norm a sublayer's output
    only): ``add_and_norm`` adds what is pending into the float32 stream and writes the stream, rounded once to the compute
    type, to ``out``.  It has no tensors."""

    def __init__(self, *, size: int, prefix: str = "") -> None:
        self.size = size

    def add_and_norm(self, residual: torch.Tensor, delta, out: torch.Tensor,
                     rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        if isinstance(delta, StreamVector):
            kernels.add_bias(residual, delta.vector)
            delta = None
        if delta is None:
            kernels.postnorm_add_rmsnorm(residual, None, None, 0.0, None, 0.0, out, rows)
        elif isinstance(delta, PostNormed):
            kernels.postnorm_add_rmsnorm(residual, delta.x, delta.weight, delta.eps, None, 0.0, out, rows, post_scale=delta.scale)
        else:
            raise TypeError("the identity norm adds nothing, or an output that passes a norm of its own")
        return out


@register_norm("layer")
class LayerNorm(Part):
    """Layer norm with weight and bias (``name`` and ``name + bias_suffix``), statistics in float32."""

    def __init__(self, *, name: str, size: int, eps: float, prefix: str = "", bias_suffix: str = ".b") -> None:
        self.name, self.bias_name, self.size, self.eps = prefix + name, prefix + name + bias_suffix, size, float(eps)
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None

    def param_specs(self) -> list[ParamSpec]:
        return [ParamSpec(self.name, (self.size,), "vector"), ParamSpec(self.bias_name, (self.size,), "vector")]

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        self.weight, self.bias = tensors[self.name], tensors[self.bias_name]
        if self.weight.dtype != self.bias.dtype:
            self.weight, self.bias = self.weight.float(), self.bias.float()

    @staticmethod
    def _pending(delta) -> tuple:
        """(first output, second output, vector) of what is still to be added to the stream."""
        if isinstance(delta, StreamVector):
            return None, None, delta.vector
        if delta is None or isinstance(delta, torch.Tensor):
            return delta, None, None
        if isinstance(delta, tuple):
            return delta[0], delta[1], None
        raise TypeError(f"the layer norm adds outputs or a vector, not {type(delta).__name__}")

    def add_and_norm(self, residual: torch.Tensor, delta, out: torch.Tensor,
                     rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``residual += delta`` (float32, in place), ``out = norm(residual)``, as :meth:`RMSNorm.add_and_norm`."""
        first, second, vector = self._pending(delta)
        kernels.add_layernorm(residual, first, self.weight, self.bias, self.eps, out, rows, second, vector)
        return out

    def shares_statistics_with(self, other) -> bool:
        """Whether :meth:`add_and_norm_both` can run this norm and ``other`` on the same stream in one kernel."""
        return isinstance(other, LayerNorm) and other.eps == self.eps and other.weight.dtype == self.weight.dtype

    def add_and_norm_both(self, residual: torch.Tensor, delta, out: torch.Tensor, other: "LayerNorm", other_out: torch.Tensor) -> None:
        first, second, vector = self._pending(delta)
        kernels.add_layernorm(residual, first, self.weight, self.bias, self.eps, out, None, second, vector, other.weight, other.bias,
                              other_out)


@register_norm("dynamic_tanh")
class DynamicTanh(Part):
    """``weight * tanh(alpha * x) + bias`` (``name``, ``name + alpha_suffix`` without dimensions, ``name + bias_suffix``), in float32."""

    def __init__(self, *, name: str, size: int, prefix: str = "", alpha_suffix: str = ".alpha", bias_suffix: str = ".b") -> None:
        self.name, self.size = prefix + name, size
        self.alpha_name, self.bias_name = self.name + alpha_suffix, self.name + bias_suffix
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None
        self.alpha = 0.0

    def param_specs(self) -> list[ParamSpec]:
        return [ParamSpec(self.name, (self.size,), "vector"), ParamSpec(self.bias_name, (self.size,), "vector"),
                ParamSpec(self.alpha_name, (), "vector")]

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        self.weight, self.bias = tensors[self.name].float().contiguous(), tensors[self.bias_name].float().contiguous()
        self.alpha = float(tensors[self.alpha_name])

    def add_and_norm(self, residual: torch.Tensor, delta, out: torch.Tensor,
                     rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``residual += delta`` (float32, in place), ``out = norm(residual)``, as :meth:`RMSNorm.add_and_norm`."""
        second = None
        if isinstance(delta, StreamVector):
            kernels.add_bias(residual, delta.vector)
            delta = None
        if isinstance(delta, tuple):
            delta, second = delta
        if delta is not None and not isinstance(delta, torch.Tensor):
            raise TypeError(f"the dynamic tanh norm adds outputs or a vector, not {type(delta).__name__}")
        kernels.add_dynamic_tanh(residual, delta, self.alpha, self.weight, self.bias, out, rows, second)
        return out
