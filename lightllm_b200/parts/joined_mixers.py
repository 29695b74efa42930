"""Several mixers side by side on one input, their outputs summed with weights, normed or as they are."""
from __future__ import annotations

import math
from typing import List, Optional, Sequence

import torch

from ..cache import CacheSpec, StateSpec
from ..config import PartSpec, part_class, register_part
from ..csrc import ops
from ..weights import WeightSpec
from . import linear as L
from .base import CacheView, LazyNorm, Mixer, Part


class JoinedMixers(Mixer):
    """``y = sum_i weight_i * rmsnorm(mixer_i(x)) * w_i``: every mixer reads the same x; each output is normed over the
    model width (``eps`` inside the root, its own plain weight ``out_norms[i]``, a full tensor name) before the sum;
    ``weights`` default to ``1 / len(mixers)`` (the mean).  ``out_norms=None``: the outputs are summed without norms, each mixer
    adding its share into the stream itself.

    Where all mixers can run from a contraction of x (``Mixer.input_weight``), the matrices are laid side by side and one
    contraction serves them all.

    At most one of the mixers may keep pages (the run has one cache plane); their fixed-size states lie one behind the
    other in the run's state plane (flat float32), each mixer finding its own at ``CacheView.state_offset``.  The
    outputs, their norms and the sum are float32."""

    graph_safe = True
    accepts_lazy_norm = False

    def __init__(self, prefix: str, hidden_size: int, mixers: Sequence[PartSpec], out_norms: Optional[Sequence[str]],
                 eps: float, weights: Optional[Sequence[float]] = None):
        if not mixers or (out_norms is not None and len(out_norms) != len(mixers)):
            raise ValueError("joined mixers: one norm weight's name for every mixer, at least one mixer")
        self.prefix, self.hidden_size, self.eps = prefix, hidden_size, float(eps)
        self.mixers: List[Mixer] = [part_class("mixer", m.kind)(m.prefix, **m.params) for m in mixers]
        self.out_names = list(out_norms) if out_norms is not None else None
        self.weights = [float(w) for w in weights] if weights is not None else [1.0 / len(mixers)] * len(mixers)
        if len(self.weights) != len(self.mixers):
            raise ValueError("joined mixers: one weight for every mixer")
        if self.out_names is None:
            for m, w in zip(self.mixers, self.weights):
                if m.takes_out_scale:
                    m.out_scale = w
        specs = [m.cache_spec() for m in self.mixers]
        paged = [i for i, s in enumerate(specs) if s is not None and s.kv is not None]
        if len(paged) > 1:
            raise ValueError("joined mixers: at most one of them may keep pages (a run has one cache plane)")
        self._kv = specs[paged[0]].kv if paged else None
        self._paged = paged[0] if paged else None
        self._offsets, total = [], 0
        for s in specs:
            self._offsets.append(total)
            if s is not None and s.state is not None:
                if s.state.dtype != "float32":
                    raise ValueError("joined mixers share one float32 state plane")
                total += math.prod(s.state.shape)
        self._state_floats = total
        self.out_w: Optional[torch.Tensor] = None           # [mixers, hidden] the norms' weights times the branches' weights
        self.w_in: Optional[torch.Tensor] = None            # the mixers' input matrices one below the other
        self.in_offsets: List[int] = []

    def children(self) -> List[Part]:
        return list(self.mixers)

    def cache_spec(self) -> Optional[CacheSpec]:
        if self._kv is None and not self._state_floats:
            return None
        return CacheSpec(kv=self._kv, state=StateSpec((self._state_floats,), "float32") if self._state_floats else None)

    def weight_specs(self) -> List[WeightSpec]:
        return [WeightSpec(n, (self.hidden_size,), init=("one_plus_normal", 0.1)) for n in self.out_names or ()]

    def bind(self, tensors, dtype, device) -> None:
        if self.out_names is not None:
            self.out_w = torch.stack([tensors[n].float() * w for n, w in zip(self.out_names, self.weights)]).contiguous()

    def bound(self) -> None:
        ws = [m.input_weight() for m in self.mixers]
        if len(ws) < 2 or any(w is None or w.dtype != ws[0].dtype for w in ws):
            return
        self.w_in = torch.cat(ws, dim=0).contiguous()
        at = 0
        for m, w in zip(self.mixers, ws):
            self.in_offsets.append(at)
            at += w.shape[0]
            m.share_input()

    def _view(self, i: int, cache: Optional[CacheView]) -> Optional[CacheView]:
        return None if cache is None else cache.at(self._offsets[i], pages=i == self._paged)

    def prepare(self, ctx, cache=None) -> None:
        for i, m in enumerate(self.mixers):
            if getattr(type(m), "prepare", None) is not Part.prepare:
                m.prepare(ctx, self._view(i, cache))

    def forward(self, x, residual, ctx, cache: Optional[CacheView]) -> None:
        if isinstance(x, LazyNorm):
            x = x.materialize()
        fused = L.linear(x, self.w_in, None, L.STORE) if self.w_in is not None else None
        n = len(self.mixers)
        branches = None
        if self.out_names is not None:
            branches = torch.zeros((n, *residual.shape), dtype=torch.float32, device=residual.device)
        for i, m in enumerate(self.mixers):
            target = branches[i] if branches is not None else residual
            apart = branches is None and not m.takes_out_scale and self.weights[i] != 1.0
            if apart:          # a mixer that cannot scale what it adds: a buffer of its own
                target = torch.zeros_like(residual)
            if fused is not None:
                m.forward_from(fused, self.in_offsets[i], target, ctx, self._view(i, cache))
            else:
                m.forward(x, target, ctx, self._view(i, cache))
            if apart:
                ops.axpy(target, residual, self.weights[i])
        if branches is None:
            return
        if n <= ops.RMSNORM_SUM_MAX:
            ops.rmsnorm_sum(branches, self.out_w, self.eps, residual)
        else:
            for i in range(n):
                ops.rmsnorm_add(branches[i], self.out_w[i], self.eps, residual, 1.0)


register_part("mixer", "joined_mixers", JoinedMixers)
