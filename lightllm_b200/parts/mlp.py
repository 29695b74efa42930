"""Dense feed-forward parts."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..config import register_part
from ..csrc import ops
from ..weights import WeightSpec
from . import linear as L
from .base import FeedForward, LazyNorm


# activation name -> the kernels' code
ACTIVATIONS = {"silu": 0, "clamped_swish": 1, "gelu_tanh": 2}


class GatedMLP(FeedForward):
    """A gated feed-forward ``h += act(x Wg^T, x Wu^T) Wd^T``.

    ``silu``: SwiGLU, ``silu(g) * u`` (src/engine/engine_server.cpp:1875-1880, SiLU as src/ops/elementwise.cu:27-33).
    ``clamped_swish``: ``g' = min(g, limit)``, ``u' = clamp(u, -limit, limit)``, ``g' * sigmoid(alpha * g') * (u' + up_shift)``.
    ``gelu_tanh``: ``0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3))) * u``.

    The gate and up matrices are interleaved row by row at load time, so that one contraction
    produces each (gate, up) pair in adjacent columns and the epilogue writes only
    ``silu(gate) * up``; the down projection adds into the residual stream in its epilogue."""

    graph_safe = True

    def __init__(self, prefix: str, hidden_size: int, intermediate_size: int, activation: str = "silu",
                 bias: bool = False, names: Optional[Dict[str, str]] = None, weight_suffix: str = ".weight",
                 alpha: float = 1.0, limit: Optional[float] = None, up_shift: float = 0.0):
        if activation not in ACTIVATIONS:
            raise ValueError(f"the gated feed-forward implements {sorted(ACTIVATIONS)}, not {activation!r}")
        if activation == "clamped_swish" and (limit is None or not limit > 0):
            raise ValueError("the clamped gate needs a positive 'limit'")
        self.prefix, self.hidden_size, self.intermediate_size, self.bias = prefix, hidden_size, intermediate_size, bias
        self.activation, self.alpha, self.limit, self.up_shift = activation, float(alpha), float(limit or 0.0), float(up_shift)
        self.names = {"gate": "gate_proj", "up": "up_proj", "down": "down_proj"}
        self.names.update(names or {})
        self.weight_suffix = weight_suffix
        self.w_gate_up = self.b_gate_up = self.w_down = self.b_down = None

    def _n(self, which: str, what: str) -> str:
        base = f"{self.prefix}.{self.names[which]}"
        return base + self.weight_suffix if what == "weight" else f"{base}.{what}"

    def weight_specs(self) -> List[WeightSpec]:
        D, I = self.hidden_size, self.intermediate_size
        specs = [WeightSpec(self._n("gate", "weight"), (I, D)), WeightSpec(self._n("up", "weight"), (I, D)),
                 WeightSpec(self._n("down", "weight"), (D, I))]
        if self.bias:
            specs += [WeightSpec(self._n("gate", "bias"), (I,)), WeightSpec(self._n("up", "bias"), (I,)),
                      WeightSpec(self._n("down", "bias"), (D,))]
        return specs

    def bind(self, tensors, dtype, device) -> None:
        g, u = tensors[self._n("gate", "weight")], tensors[self._n("up", "weight")]
        wdt = torch.float32 if torch.float32 in (g.dtype, u.dtype) else g.dtype
        I, D = g.shape
        self.w_gate_up = torch.stack([g.to(wdt), u.to(wdt)], dim=1).reshape(2 * I, D).contiguous()
        self.w_down = tensors[self._n("down", "weight")]
        L.reserve_fused_scratch(device, 2 * I)
        if self.bias:
            bg, bu = tensors[self._n("gate", "bias")].float(), tensors[self._n("up", "bias")].float()
            self.b_gate_up = torch.stack([bg, bu], dim=1).reshape(2 * I).contiguous()
            self.b_down = tensors[self._n("down", "bias")].float().contiguous()

    accepts_lazy_norm = True

    def forward(self, x, residual, ctx=None) -> None:
        if self.activation != "silu":
            if isinstance(x, LazyNorm):
                x = x.materialize()
            act = L.linear_glu(x, self.w_gate_up, self.b_gate_up, ACTIVATIONS[self.activation], self.alpha, self.limit,
                               self.up_shift)
            L.linear(act, self.w_down, self.b_down, L.RESIDUAL, residual=residual)
            return
        if isinstance(x, LazyNorm):
            act = L.linear_normed(x, self.w_gate_up, self.b_gate_up, L.SWIGLU)
        else:
            act = L.linear(x, self.w_gate_up, self.b_gate_up, L.SWIGLU)
        L.linear(act, self.w_down, self.b_down, L.RESIDUAL, residual=residual)


# activation name of a feed-forward without a gate -> the code of the contractions' store epilogue
PLAIN_ACTIVATIONS = {"squared_relu": ops.ACT_SQUARED_RELU}


class PlainMLP(FeedForward):
    """A feed-forward without a gate, ``h += act(x Wu^T) Wd^T``; ``squared_relu``: ``max(z, 0)^2``.  The activation is taken in the
    epilogue of the first contraction, from its float accumulators; no biases."""

    graph_safe = True

    def __init__(self, prefix: str, hidden_size: int, intermediate_size: int, activation: str = "squared_relu",
                 names: Optional[Dict[str, str]] = None, weight_suffix: str = ".weight"):
        if activation not in PLAIN_ACTIVATIONS:
            raise ValueError(f"the plain feed-forward implements {sorted(PLAIN_ACTIVATIONS)}, not {activation!r}")
        self.hidden_size, self.intermediate_size, self.activation = hidden_size, intermediate_size, activation
        names = {"up": "up_proj", "down": "down_proj", **(names or {})}
        self.up_name, self.down_name = (f"{prefix}.{names[n]}{weight_suffix}" for n in ("up", "down"))
        self.w_up = self.w_down = None

    def weight_specs(self) -> List[WeightSpec]:
        D, I = self.hidden_size, self.intermediate_size
        return [WeightSpec(self.up_name, (I, D)), WeightSpec(self.down_name, (D, I))]

    def bind(self, tensors, dtype, device) -> None:
        self.w_up, self.w_down = tensors[self.up_name], tensors[self.down_name]

    def forward(self, x, residual, ctx=None) -> None:
        if isinstance(x, LazyNorm):
            x = x.materialize()
        act = L.linear(x, self.w_up, None, L.STORE, glu=(PLAIN_ACTIVATIONS[self.activation], 1.0, 0.0, 0.0))
        L.linear(act, self.w_down, None, L.RESIDUAL, residual=residual)


register_part("ffn", "gated_mlp", GatedMLP)
register_part("ffn", "plain_mlp", PlainMLP)
