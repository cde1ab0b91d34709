"""Gated feed-forward: down( act(gate(h)) * up(h) ) with gate and up as one matrix; or the capped form down( g
sigmoid(1.702 g) (u + 1) ) with g = min(gate(h), limit), u = clamp(up(h), -limit, limit).  act is silu or the tanh form of gelu;
with ``bias`` all three projections have one.

pico_vllm/model.py:309-318 (fused gate_up projection, silu(gate) * up, down projection);
the activation runs in float32 as in pico_vllm/kernels/swiglu.py:28-44.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from ..errors import ConfigError
from .base import Param, Part, Piece
from .registry import register


@register("feed_forward", "gated_mlp")
class GatedMLP(Part):
    fuses_residual = True   # forward(..., residual=x) may add its output to x and return None

    def __init__(self, width: int, inner: int, act: str = "silu", limit: Optional[float] = None, bias: bool = False):
        if act not in ("silu", "capped", "gelu_tanh"):
            raise ConfigError(f"gated_mlp: activation {act!r} is not built (only 'silu', 'capped' and 'gelu_tanh')")
        if bias and act == "capped":
            raise ConfigError("gated_mlp: biases are not built with the capped activation")
        if (act == "capped") != bool(limit and limit > 0):
            raise ConfigError("gated_mlp: the capped activation, and it alone, needs a positive limit")
        self.width, self.inner, self.act = width, inner, act
        self.limit = float(limit) if limit else None
        self.has_bias = bias
        self.gate_up_weight = self.down_weight = self.gate_up_bias = self.down_bias = self.down_bias_act = None

    def params(self) -> List[Param]:
        ps = [Param("gate_up_weight", (Piece("gate.weight", (self.inner, self.width)),
                                       Piece("up.weight", (self.inner, self.width)))),
              Param("down_weight", (Piece("down.weight", (self.width, self.inner)),))]
        if self.has_bias:
            ps += [Param("gate_up_bias", (Piece("gate.bias", (self.inner,)), Piece("up.bias", (self.inner,))), kind="vector"),
                   Param("down_bias", (Piece("down.bias", (self.width,)),), kind="vector")]
        return ps

    def materialize(self, device, dtype):
        if self.down_bias is not None:
            self.down_bias_act = self.down_bias.to(dtype)

    def can_fuse_norm(self, x: torch.Tensor, norm) -> bool:
        return self.act != "gelu_tanh" and not self.has_bias and getattr(norm, "plain_rms", False) and getattr(norm, "weight", None) is not None and self.inner % 8 == 0 \
            and ops.skinny_norm_takes(x, self.gate_up_weight)

    def forward(self, h: Optional[torch.Tensor], batch, residual: Optional[torch.Tensor] = None, norm=None):
        """Returns what is to be added to the residual stream - or, when ``residual`` is given
        and the fused small-batch kernels take the sizes, adds it there itself and returns None.
        With ``norm`` (after ``can_fuse_norm``), ``h`` is None and the normed input is computed from
        ``residual`` inside the first kernel."""
        if self.has_bias or self.act == "gelu_tanh":
            return self._forward_biased(h)
        if norm is not None:
            a = ops.skinny_gate_up_swiglu(residual, self.gate_up_weight, norm.weight, norm.eps, limit=self.limit)
        elif ops.skinny_takes(h, self.gate_up_weight) and self.inner % 8 == 0:
            a = ops.skinny_gate_up_swiglu(h, self.gate_up_weight, limit=self.limit)      # product and activation in one kernel
        elif h.shape[0] >= ops.TC_PAIR_MIN_TOKENS and ops.tc_takes(h, self.gate_up_weight) and self.inner % 8 == 0:
            # many tokens: tcgen05 product with the activation in its epilogue (the [T, 2I] buffer never exists);
            # below that the library product and the activation kernel are faster (measured, see ops)
            a = ops.tc_gate_up_swiglu(h, self.gate_up_weight, limit=self.limit)
        else:
            gu = ops.linear(h, self.gate_up_weight)
            if self.limit:
                a = ops.capped_glu(gu, self.inner, self.limit)
            else:
                a = torch.empty((h.shape[0], self.inner), dtype=h.dtype, device=h.device)
                ops.swiglu(gu, a)
        if residual is not None and ops.skinny_takes(a, self.down_weight):
            ops.skinny_linear_residual(a, self.down_weight, residual)
            return None
        if ops.skinny_takes(a, self.down_weight):
            return ops.skinny_linear(a, self.down_weight)
        return ops.linear(a, self.down_weight)

    def _forward_biased(self, h: torch.Tensor) -> torch.Tensor:
        """The form with biases, or with the tanh form of gelu: the activation and the biases in the first product's epilogue
        (gelu), or in one kernel behind it; the last bias in the epilogue of the down product."""
        if self.act == "gelu_tanh" and self.inner % 8 == 0 and ops.skinny_takes(h, self.gate_up_weight):
            a = ops.skinny_gate_up_gelu(h, self.gate_up_weight, self.gate_up_bias)
        elif self.act == "gelu_tanh" and self.inner % 8 == 0 and h.shape[0] >= ops.TC_PAIR_MIN_TOKENS and ops.tc_takes(h, self.gate_up_weight):
            a = ops.tc_gate_up_gelu(h, self.gate_up_weight, self.gate_up_bias)
        else:
            a = ops.bias_glu(ops.linear(h, self.gate_up_weight), self.gate_up_bias, self.act)
        if self.has_bias:
            return ops.linear_bias(a, self.down_weight, self.down_bias, self.down_bias_act)
        return ops.skinny_linear(a, self.down_weight) if ops.skinny_takes(a, self.down_weight) else ops.linear(a, self.down_weight)
