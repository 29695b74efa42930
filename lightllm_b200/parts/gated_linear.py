"""Gated linear attention: a recurrence over a per-request state with a decay per key channel and token."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..cache import CacheSpec, StateSpec
from ..config import register_part
from ..csrc import ops
from ..weights import WeightSpec
from . import linear as L
from .base import CacheView, LazyNorm, Mixer
from .conv_attention import span_arrays
from .retention import recurrence_pieces


class GatedLinearMixer(Mixer):
    """Per head, with a state ``S [head_dim, v_head_dim]`` that is zero before a request's first token::

        S <- diag(alpha_t) S + k_t v_t^T;   o_t = S^T (q_scale q_t)          alpha = sigmoid(W_a2 (W_a1 x) + b)^(1 / tau)
        out = W_o ((o / rms(o) over a head * w) * silu(W_g x))

    ``q_scale`` defaults to ``head_dim ** -0.5``; the norm's weight [v_head_dim] is shared by the heads.  One contraction makes
    everything that reads x (q | k | v | gate | the decay's low-rank input).  The state lives in float32 in the request's
    slot, so the result does not depend on how the tokens were cut; the decays' logarithms, the recurrence, the norm and the
    gate are float32 in both precisions."""

    graph_safe = True
    accepts_lazy_norm = False
    takes_out_scale = True

    def __init__(self, prefix: str, hidden_size: int, num_heads: int, head_dim: int, v_head_dim: int, decay_rank: int, tau: float,
                 q_scale: Optional[float] = None, norm_eps: float = 1e-6, names: Optional[Dict[str, str]] = None,
                 weight_suffix: str = ".weight", bias_ending: str = "bias"):
        if not tau > 0:
            raise ValueError(f"the decays' root tau must be positive, got {tau}")
        self.prefix, self.hidden_size = prefix, hidden_size
        self.num_heads, self.head_dim, self.v_head_dim, self.decay_rank = num_heads, head_dim, v_head_dim, int(decay_rank)
        self.tau, self.norm_eps = float(tau), float(norm_eps)
        self.q_scale = float(q_scale) if q_scale is not None else head_dim ** -0.5
        self.names = {"q": "q_proj", "k": "k_proj", "v": "v_proj", "g": "g_proj", "o": "o_proj", "a1": "a_down", "a2": "a_up",
                      "norm": "norm"}
        self.names.update(names or {})
        self.weight_suffix, self.bias_ending = weight_suffix, bias_ending
        self.w_fused = self.w_a2 = self.b_a2 = self.norm_w = self.w_o = None

    def _n(self, which: str, ending: Optional[str] = None) -> str:
        base = f"{self.prefix}.{self.names[which]}"
        return base + self.weight_suffix if ending is None else f"{base}.{ending}" if ending else base

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(state=StateSpec((self.num_heads * self.head_dim * self.v_head_dim,), "float32"))

    def weight_specs(self) -> List[WeightSpec]:
        D, H, hd, vd, r = self.hidden_size, self.num_heads, self.head_dim, self.v_head_dim, self.decay_rank
        return [WeightSpec(self._n("q"), (H * hd, D)), WeightSpec(self._n("k"), (H * hd, D)), WeightSpec(self._n("v"), (H * vd, D)),
                WeightSpec(self._n("g"), (H * vd, D)), WeightSpec(self._n("a1"), (r, D)),
                WeightSpec(self._n("a2"), (H * hd, r), init=("normal", 0.2)),
                WeightSpec(self._n("a2", self.bias_ending), (H * hd,), init=("normal", 1.0)),
                WeightSpec(self._n("norm", ""), (vd,), init=("one_plus_normal", 0.1)), WeightSpec(self._n("o"), (D, H * vd))]

    def bind(self, tensors, dtype, device) -> None:
        ws = [tensors[self._n(p)] for p in ("q", "k", "v", "g", "a1")]
        wdt = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
        pad = -sum(w.shape[0] for w in ws) % 8          # whole 16-byte pieces a row of the fused output
        if pad:
            ws.append(torch.zeros((pad, self.hidden_size), dtype=wdt, device=ws[0].device))
        self.w_fused = torch.cat([w.to(wdt) for w in ws], dim=0).contiguous()
        self.w_a2 = tensors[self._n("a2")].contiguous()
        self.b_a2 = tensors[self._n("a2", self.bias_ending)].float().contiguous()
        self.norm_w = tensors[self._n("norm", "")].float().contiguous()
        self.w_o = tensors[self._n("o")]

    @property
    def prepare_key(self):
        return ("gated_linear", self.num_heads, self.head_dim, self.v_head_dim)

    def prepare(self, ctx, cache=None) -> None:
        recurrence_pieces(ctx, self.num_heads, self.head_dim, self.v_head_dim)

    def input_weight(self) -> Optional[torch.Tensor]:
        return self.w_fused

    def share_input(self) -> None:
        self.w_fused = None

    def forward(self, x, residual, ctx, cache: CacheView) -> None:
        if isinstance(x, LazyNorm):
            x = x.materialize()
        self.forward_from(L.linear(x, self.w_fused, None, L.STORE), 0, residual, ctx, cache)

    def forward_from(self, fused, offset: int, residual, ctx, cache: CacheView) -> None:
        """``fused`` [T, ..]: q | k | v | gate | decay input from column ``offset`` on."""
        if cache is None or cache.state is None or not cache.writes:
            raise ops.KernelError("gated linear attention: the run needs a state plane of its own (the recurrence advances it)")
        T = fused.shape[0]
        H, hd, vd = self.num_heads, self.head_dim, self.v_head_dim
        f32 = dict(dtype=torch.float32, device=fused.device)
        v0 = offset + 2 * H * hd
        g0 = v0 + H * vd
        decay = torch.empty((T, H * hd), **f32)
        ops.low_rank_up(fused, g0 + H * vd, self.w_a2, decay, bias=self.b_a2, mode="log_sigmoid", multiplier=1.0 / self.tau)
        o = torch.empty((T, H * vd), **f32)
        ops.gated_linear(fused, offset, offset + H * hd, v0, decay, self.q_scale, span_arrays(ctx), H, hd, vd, cache.state,
                         cache.state_offset, o, pieces=recurrence_pieces(ctx, H, hd, vd))
        gated = torch.empty((T, H * vd), dtype=fused.dtype, device=fused.device)
        ops.head_gate(o, fused[:, g0: g0 + H * vd], gated, H, vd, False, "silu", unit_rms=True, eps=self.norm_eps,
                      norm_weight=self.norm_w)
        L.linear(gated, self.w_o, None, L.RESIDUAL, residual=residual, scale=self.out_scale)


register_part("mixer", "gated_linear_attention", GatedLinearMixer)
