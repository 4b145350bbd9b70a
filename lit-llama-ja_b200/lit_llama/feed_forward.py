"""Dense feed-forward layers of the folder-loaded models: ``W_down act(W_up h)`` or, gated, ``W_down (silu(W_gate h) * (W_up h))``,
with the activation as a parameter."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn
from torch.nn import functional as F

from . import _native as N


def glu_unit(gu: torch.Tensor, ff: int, limit: float = float("inf"), alpha: float = 1.0, shift: float = 0.0,
             bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``gu [rows, >= 2 ff]`` (columns [gate | up | ...]) -> ``[rows, ff]``: ``g * sigmoid(alpha * g) * (u + shift)`` with
    ``g = min(gate, limit)`` and ``u = clamp(up, -limit, limit)``; the defaults are the plain silu-gated unit.  ``bias`` (fp32
    ``[2 ff]``) joins [gate | up] first; ``out``: a column slice to write to."""
    if out is None:
        out = torch.empty((gu.shape[0], ff), dtype=gu.dtype, device=gu.device)
    N.call("ll_glu_unit_rows", N.ptr(gu), gu.stride(0), ff, N.ptr(bias), float(limit), float(alpha), float(shift), N.ptr(out), out.stride(0),
           N.dtype_code(gu.dtype), gu.shape[0], N.stream())
    return out


def relu_squared_(h: torch.Tensor) -> torch.Tensor:
    """``relu(h)^2``, in place."""
    N.call("ll_relu_squared", N.ptr(h), N.dtype_code(h.dtype), h.numel(), N.stream())
    return h


class DenseFF(nn.Module):
    """``act``: "relu2" (the square of relu), "gelu" (the erf form), "gelu_tanh" or "silu_glu" (silu-gated; the gate and up
    projections are one GEMM over their stacked weights)."""

    def __init__(self, width: int, ff: int, act: str, dtype: torch.dtype, device) -> None:
        super().__init__()
        if act not in ("relu2", "gelu", "gelu_tanh", "silu_glu"):
            raise ValueError(f"unknown feed-forward activation {act!r}")
        self.act, self.ff = act, ff
        kw = dict(dtype=dtype, device=device)
        rows = (2 * ff + 7) // 8 * 8 if act == "silu_glu" else ff          # [gate; up], zero rows up to a multiple of 8
        self.w_up = nn.Parameter(torch.zeros((rows, width), **kw), requires_grad=False)
        self.w_down = nn.Parameter(torch.zeros((width, ff), **kw), requires_grad=False)

    def load(self, get) -> None:
        if self.act == "silu_glu":
            self.w_up.zero_()
            self.w_up[: self.ff].copy_(get("gate"))
            self.w_up[self.ff: 2 * self.ff].copy_(get("up"))
        else:
            self.w_up.copy_(get("up"))
        self.w_down.copy_(get("down"))

    def forward(self, x_act: torch.Tensor) -> torch.Tensor:
        h = F.linear(x_act, self.w_up)
        if self.act == "silu_glu":
            h = glu_unit(h, self.ff)
        elif self.act == "relu2":
            relu_squared_(h)
        else:
            N.call("ll_gelu", N.ptr(h), N.dtype_code(h.dtype), 1 if self.act == "gelu_tanh" else 0, h.numel(), N.stream())
        return F.linear(h, self.w_down)


class ClampedUnit(nn.Module):
    """The element-wise part of a gated feed-forward whose projections have biases and whose unit is clamped,
    ``z = unit([gate | up] + b)``, ``y = W_down z + b_down``.  The projections themselves belong to the layer, which stacks
    them with those of the sublayer that reads the same input; ``in_rows`` and ``down`` hand over what it stacks."""

    def __init__(self, width: int, ff: int, limit: float, device, alpha: float = 1.702, shift: float = 1.0) -> None:
        super().__init__()
        f32 = dict(dtype=torch.float32, device=device)
        self.ff, self.limit, self.alpha, self.shift = ff, float(limit), float(alpha), float(shift)
        self.bias = nn.Parameter(torch.zeros(2 * ff, **f32), requires_grad=False)            # [gate | up]
        self.bias_down = nn.Parameter(torch.zeros(width, **f32), requires_grad=False)

    def in_rows(self, get) -> torch.Tensor:
        return torch.cat([get("gate"), get("up")], dim=0)

    def down(self, get) -> torch.Tensor:
        return get("down")

    def load(self, get) -> None:
        self.bias[: self.ff].copy_(get("gate.b").float())
        self.bias[self.ff:].copy_(get("up.b").float())
        self.bias_down.copy_(get("down.b").float())

    def forward(self, gu: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        return glu_unit(gu, self.ff, self.limit, self.alpha, self.shift, self.bias, out)
