"""Feed-forward parts.  ``gated_mlp``: ``down(act(gate(x)) * up(x))`` without biases
(miniserve/model/layers.py:71-87) with ``silu`` or ``gelu_tanh`` (the tanh form of GELU, no biases) as the activation, or, ``clamped_glu`` with ``limit``, ``down(g sigmoid(1.702 g) (u +
1))`` with ``g = min(gate(x), limit)`` and ``u = clamp(up(x), -limit, limit)``; gate and up run as one
matrix product over one weight that holds both.  Where the intermediate size is a multiple of eight
the rows of the two alternate in blocks of eight (``kernels.interleave_gate_up``), which lets the
product of a decode step apply the activation as it stores; else the up rows follow the gate rows.  With ``bias=True`` the
three projections have biases (``down(act(gate(x) + b_g) * (up(x) + b_u)) + b_d``, added in float32 as the activation and
the output are formed); the up rows then follow the gate rows.  ``mlp``: ``down(act(up(x)))`` without a gate and without biases,
``act`` the square of ReLU."""

from __future__ import annotations

from typing import Optional, Union

import torch

from .. import kernels
from .base import FoldedInput, NormFold, ParamSpec, Part, ResidualAdd, register_feed_forward
from .context import StepContext


@register_feed_forward("gated_mlp")
class GatedMLP(Part):
    def __init__(self, *, prefix: str, hidden_size: int, intermediate_size: int, activation: str = "silu",
                 gate_name: str = "gate_proj.weight", up_name: str = "up_proj.weight",
                 down_name: str = "down_proj.weight", bias: bool = False, limit: Optional[float] = None,
                 gate_bias_name: str = "gate_proj.bias", up_bias_name: str = "up_proj.bias", down_bias_name: str = "down_proj.bias") -> None:
        if activation not in ("silu", "clamped_glu", "gelu_tanh"):
            raise ValueError(f"gated_mlp implements the activations 'silu', 'gelu_tanh' and 'clamped_glu', not {activation!r}")
        if activation == "gelu_tanh" and bias:
            raise ValueError("gated_mlp: biases are implemented for the 'silu' activation")
        self.activation = activation
        if (activation == "clamped_glu") != (limit is not None) or (limit is not None and (limit <= 0 or bias)):
            raise ValueError(f"gated_mlp: 'clamped_glu' takes a limit above 0 and no biases, the others no limit (limit {limit}, bias {bias})")
        self.limit = None if limit is None else float(limit)
        self.hidden_size, self.intermediate_size = hidden_size, intermediate_size
        self.names = dict(gate=prefix + gate_name, up=prefix + up_name, down=prefix + down_name,
                          gate_b=prefix + gate_bias_name, up_b=prefix + up_bias_name, down_b=prefix + down_bias_name)
        self.bias = bool(bias)
        self.gate_up_bias: Optional[torch.Tensor] = None
        self.down_bias: Optional[torch.Tensor] = None
        self.gate_up_weight: Optional[torch.Tensor] = None
        self.down_weight: Optional[torch.Tensor] = None
        self.paired = False

    def param_specs(self) -> list[ParamSpec]:
        h, i = self.hidden_size, self.intermediate_size
        specs = [ParamSpec(self.names["gate"], (i, h)), ParamSpec(self.names["up"], (i, h)),
                 ParamSpec(self.names["down"], (h, i))]
        if self.bias:
            specs += [ParamSpec(self.names["gate_b"], (i,), "vector"), ParamSpec(self.names["up_b"], (i,), "vector"),
                      ParamSpec(self.names["down_b"], (h,), "vector")]
        return specs

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        gate, up = tensors[self.names["gate"]], tensors[self.names["up"]]
        self.paired = self.intermediate_size % kernels.GATE_UP_BLOCK == 0 and not self.bias
        if self.bias:
            self.gate_up_bias = torch.cat([tensors[self.names["gate_b"]].float(), tensors[self.names["up_b"]].float()]).contiguous()
            self.down_bias = tensors[self.names["down_b"]].float().contiguous()
        if self.paired:
            self.gate_up_weight = kernels.interleave_gate_up(gate, up).contiguous()
        else:
            self.gate_up_weight = torch.cat([gate, up], dim=0).contiguous()
        self.down_weight = tensors[self.names["down"]]

    # norms folded into the projections (the gate/up weight only in its interleaved form: the product that
    # completes the norm is the one that applies the activation)
    fold_input_gated = True

    def fold_input_weight(self, ctx: StepContext) -> Optional[torch.Tensor]:
        return self.gate_up_weight if self.paired else None

    def fold_output_weight(self, ctx: StepContext) -> Optional[torch.Tensor]:
        return self.down_weight if self.paired else None

    def forward(self, x, ctx: StepContext, fold: Union[None, NormFold, ResidualAdd] = None):
        """``x``: the normed input, or a :class:`FoldedInput`.  With a :class:`NormFold` the down projection adds into
        the residual stream and a :class:`FoldedInput` for the part behind the following norm is returned; with a
        :class:`ResidualAdd` it adds into the stream and nothing is returned."""
        stats = None
        if isinstance(x, FoldedInput):
            x, stats = x.x, x.stats
        n = x.shape[0]
        out = ctx.buffer("gated_mlp.out", (n, self.hidden_size), x.dtype)
        if self.paired:
            hidden = ctx.buffer("gated_mlp.hidden", (n, self.intermediate_size), x.dtype)
            kernels.gated_up(x, self.gate_up_weight, hidden, row_stats=stats, limit=self.limit, activation=self.activation)
            if isinstance(fold, ResidualAdd):
                kernels.linear_add(hidden, self.down_weight, fold.residual)
                return None
            if fold is not None:
                partials = ctx.buffer("gated_mlp.partials", kernels.residual_partials_shape(n, *self.down_weight.shape), torch.float32)
                stats = kernels.linear_residual(hidden, self.down_weight, fold.residual, fold.weight, fold.eps, out,
                                                     partials)
                return FoldedInput(out, stats)
            kernels.linear(hidden, self.down_weight, out)
        else:
            gate_up = ctx.buffer("gated_mlp.gate_up", (n, 2 * self.intermediate_size), x.dtype)
            kernels.linear(x, self.gate_up_weight, gate_up)
            if self.bias:
                hidden = ctx.buffer("gated_mlp.hidden", (n, self.intermediate_size), x.dtype)
                kernels.silu_mul(gate_up, hidden, bias=self.gate_up_bias)
                kernels.linear(hidden, self.down_weight, out)
                kernels.add_bias(out, self.down_bias)
            elif self.activation != "silu":
                hidden = ctx.buffer("gated_mlp.hidden", (n, self.intermediate_size), x.dtype)
                kernels.silu_mul(gate_up, hidden, limit=self.limit, activation=self.activation)
                kernels.linear(hidden, self.down_weight, out)
            else:
                kernels.gated_linear(gate_up, self.down_weight, out)
        return out


@register_feed_forward("mlp")
class PlainMLP(Part):
    def __init__(self, *, prefix: str, hidden_size: int, intermediate_size: int, activation: str = "relu_square",
                 up_name: str = "up", down_name: str = "down") -> None:
        if activation != "relu_square":
            raise ValueError(f"mlp implements the 'relu_square' activation, not {activation!r}")
        self.hidden_size, self.intermediate_size = hidden_size, intermediate_size
        self.names = dict(up=prefix + up_name, down=prefix + down_name)
        self.up_weight: Optional[torch.Tensor] = None
        self.down_weight: Optional[torch.Tensor] = None

    def param_specs(self) -> list[ParamSpec]:
        return [ParamSpec(self.names["up"], (self.intermediate_size, self.hidden_size)),
                ParamSpec(self.names["down"], (self.hidden_size, self.intermediate_size))]

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        self.up_weight, self.down_weight = tensors[self.names["up"]], tensors[self.names["down"]]

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        n = x.shape[0]
        hidden = ctx.buffer("mlp.hidden", (n, self.intermediate_size), x.dtype)
        kernels.linear(x, self.up_weight, hidden)
        kernels.relu_square(hidden)
        out = ctx.buffer("mlp.out", (n, self.hidden_size), x.dtype)
        kernels.linear(hidden, self.down_weight, out)
        return out
