"""Attention whose scores lose a bias by distance: no positions but the distance between query and key."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..config import register_part
from ..csrc import ops
from ..weights import WeightSpec
from . import linear as L
from .attention import AttentionMixer
from .base import CacheView, LazyNorm


def geometric_slopes(heads: int) -> List[float]:
    """``2^(-8 (h + 1) / heads)`` for head h."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


class DistanceAttentionMixer(AttentionMixer):
    """Grouped-query attention in which position enters the scores as a bias alone::

        q, k <- rms_norm(q or k over a head) * w        (``qk_norm``: a weight [head_dim] shared by the heads, ``<q>.norm``)
        s = scale q . k;  s <- softcap tanh(s / softcap)        (``softcap``; none: the scores as they are)
        s <- s - slope_h (i - j)                                slope_h = 2^(-8 (h + 1) / heads)
        p = exp(s) / (sum over the window of exp(s) + exp(sink))        (``sink``: one number for all heads, a score without
                                                                        key, value, cap or bias; 0 adds one to the sum)

    Values may be of another width than the keys; ``window`` and ``keep_first`` as :class:`AttentionMixer`.  One contraction
    makes q, k and v, one kernel norms q and k and writes the cache rows of the new tokens."""

    graph_safe = True
    accepts_lazy_norm = False
    takes_out_scale = True

    def __init__(self, prefix: str, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int,
                 v_head_dim: Optional[int] = None, window: Optional[int] = None, keep_first: int = 0, scale: Optional[float] = None,
                 softcap: Optional[float] = None, sink: Optional[float] = None, qk_norm: bool = True, norm_eps: float = 1e-6,
                 names: Optional[Dict[str, str]] = None, weight_suffix: str = ".weight", norm_ending: str = "norm"):
        if softcap is not None and not softcap > 0:
            raise ValueError(f"a soft cap on the scores must be positive, got {softcap}")
        super().__init__(prefix, hidden_size, num_heads, num_kv_heads, head_dim, qkv_bias=False, out_bias=False, window=window,
                         scale=scale, names=names, weight_suffix=weight_suffix, v_head_dim=v_head_dim, keep_first=keep_first)
        self.softcap = float(softcap) if softcap else None
        self.sink, self.qk_norm, self.norm_eps, self.norm_ending = sink, bool(qk_norm), float(norm_eps), norm_ending
        self.w_fused = self.q_norm_w = self.k_norm_w = None

    def weight_specs(self) -> List[WeightSpec]:
        D, H, G, d, vd = self.hidden_size, self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim
        specs = [WeightSpec(self._n("q", "weight"), (H * d, D)), WeightSpec(self._n("k", "weight"), (G * d, D)),
                 WeightSpec(self._n("v", "weight"), (G * vd, D)), WeightSpec(self._n("o", "weight"), (D, H * vd))]
        if self.qk_norm:
            specs += [WeightSpec(self._n(p, self.norm_ending), (d,), init=("one_plus_normal", 0.1)) for p in "qk"]
        return specs

    def bind(self, tensors, dtype, device) -> None:
        ws = [tensors[self._n(p, "weight")] for p in "qkv"]
        wdt = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
        pad = -sum(w.shape[0] for w in ws) % 8          # whole 16-byte pieces a row of the fused output
        if pad:
            ws.append(torch.zeros((pad, self.hidden_size), dtype=wdt, device=ws[0].device))
        self.w_fused = torch.cat([w.to(wdt) for w in ws], dim=0).contiguous()
        self.w_o = tensors[self._n("o", "weight")]
        if self.qk_norm:
            self.q_norm_w, self.k_norm_w = (tensors[self._n(p, self.norm_ending)].float().contiguous() for p in "qk")
        self.slopes = torch.tensor(geometric_slopes(self.num_heads), dtype=torch.float32, device=device)
        if self.sink is not None:
            self.sinks = torch.full((self.num_heads,), float(self.sink), dtype=torch.float32, device=device)

    def input_weight(self) -> Optional[torch.Tensor]:
        return self.w_fused

    def share_input(self) -> None:
        self.w_fused = None

    def forward(self, x, residual, ctx, cache: CacheView) -> None:
        if isinstance(x, LazyNorm):
            x = x.materialize()
        self.forward_from(L.linear(x, self.w_fused, None, L.STORE), 0, residual, ctx, cache)

    def forward_from(self, fused, offset: int, residual, ctx, cache: CacheView) -> None:
        """``fused`` [T, ..]: q | k | v from column ``offset`` on."""
        T = fused.shape[0]
        H, G, d, vd = self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim
        writes = cache.writes
        q = torch.empty((T, H * d), dtype=fused.dtype, device=fused.device)
        k0 = offset + H * d
        ops.head_prepare(fused, offset, k0, H, G if writes else 0, d, ctx.positions,
                         ctx.slot_mapping[cache.group] if writes else None, q, cache.k, cache.v,
                         values="columns" if writes else None, v_off=k0 + G * d if writes else -1, v_width=G * vd if writes else 0,
                         q_norm_w=self.q_norm_w, k_norm_w=self.k_norm_w, eps=self.norm_eps)
        attn = torch.empty((T, H * vd), dtype=fused.dtype, device=fused.device)
        self.attend(q, cache, ctx, attn)
        L.linear(attn, self.w_o, None, L.RESIDUAL, residual=residual, scale=self.out_scale)


register_part("mixer", "distance_attention", DistanceAttentionMixer)
