"""The Mamba-2 mixer: a state-space recurrence with one decay a head and token over a per-request state."""
from __future__ import annotations

from typing import Dict, List, Optional

import numpy as np
import torch

from ..cache import CacheSpec, StateSpec
from ..config import register_part
from ..csrc import ops
from ..weights import WeightSpec
from . import linear as L
from .base import CacheView, LazyNorm, Mixer
from .conv_attention import span_arrays


class StateSpaceMixer(Mixer):
    """Per head, with a state ``S [state, v_head_dim]`` that is zero before a request's first token::

        [z | x | B | C | dt] = W_in h
        x, B, C <- silu(conv(.) + b)                          causal, per channel, ``conv_taps`` taps
        dt <- softplus(dt + dt_bias)
        S <- exp(-exp(A_log) dt) S + dt B x^T;   y = S^T C + D x
        out = W_o (norm(y * silu(z)) * w)

    B and C have ``groups`` vectors, shared by ``num_heads / groups`` neighbouring heads each; the norm divides each of
    ``norm_groups`` equal parts of the concatenated heads by its own root mean square (the gate comes before it).

    One contraction makes everything that reads h.  The request's state slot holds S and the convolution's inputs of the last
    ``conv_taps - 1`` positions, both float32, so the result does not depend on how the tokens were cut.  dt, decays, the
    state, y and the norm are float32 in both precisions; x, B and C leave the convolution in the compute dtype."""

    graph_safe = True
    accepts_lazy_norm = False

    def __init__(self, prefix: str, hidden_size: int, num_heads: int, v_head_dim: int, state_dim: int, groups: int,
                 conv_taps: int, norm_groups: int = 1, norm_eps: float = 1e-6, names: Optional[Dict[str, str]] = None,
                 weight_suffix: str = ".weight", bias_ending: str = "bias"):
        inner = num_heads * v_head_dim
        if num_heads % groups:
            raise ValueError(f"{num_heads} heads are not a multiple of {groups} groups")
        if inner % norm_groups:
            raise ValueError(f"{inner} channels do not fall into {norm_groups} equal parts")
        if conv_taps < 1:
            raise ValueError(f"a convolution has at least one tap, got {conv_taps}")
        self.prefix, self.hidden_size = prefix, hidden_size
        self.num_heads, self.v_head_dim, self.state_dim, self.groups = num_heads, v_head_dim, state_dim, groups
        self.conv_taps, self.norm_groups, self.norm_eps = int(conv_taps), int(norm_groups), float(norm_eps)
        self.inner, self.channels = inner, inner + 2 * groups * state_dim          # channels: what the convolution sees
        self.names = {"in": "in_proj", "conv": "conv1d", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D", "norm": "norm",
                      "o": "out_proj"}
        self.names.update(names or {})
        self.weight_suffix, self.bias_ending = weight_suffix, bias_ending
        self.state_floats = num_heads * state_dim * v_head_dim
        self.w_in = self.w_conv = self.b_conv = self.dt_bias = self.rate = self.skip = self.norm_w = self.w_o = None

    def _n(self, which: str, ending: Optional[str] = None) -> str:
        base = f"{self.prefix}.{self.names[which]}"
        return base + self.weight_suffix if ending is None else f"{base}.{ending}" if ending else base

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(state=StateSpec((self.state_floats + (self.conv_taps - 1) * self.channels,), "float32"))

    def weight_specs(self) -> List[WeightSpec]:
        D, H = self.hidden_size, self.num_heads
        return [WeightSpec(self._n("in"), (self.inner + self.channels + H, D)),
                WeightSpec(self._n("conv"), (self.channels, self.conv_taps), init=("normal", 0.5)),
                WeightSpec(self._n("conv", self.bias_ending), (self.channels,), init=("normal", 0.1)),
                WeightSpec(self._n("dt_bias", ""), (H,), init=("normal", 0.5)),
                WeightSpec(self._n("A_log", ""), (H,), init=("normal", 0.5)),
                WeightSpec(self._n("D", ""), (H,), init=("one_plus_normal", 0.1)),
                WeightSpec(self._n("norm", ""), (self.inner,), init=("one_plus_normal", 0.1)),
                WeightSpec(self._n("o"), (D, self.inner))]

    def bind(self, tensors, dtype, device) -> None:
        w = tensors[self._n("in")]
        pad = -w.shape[0] % 8          # whole 16-byte pieces a row of the projection's output
        self.w_in = torch.cat([w, w.new_zeros((pad, w.shape[1]))], dim=0).contiguous() if pad else w
        self.w_conv = tensors[self._n("conv")].float().contiguous()
        self.b_conv = tensors[self._n("conv", self.bias_ending)].float().contiguous()
        self.dt_bias = tensors[self._n("dt_bias", "")].float().contiguous()
        self.rate = torch.exp(tensors[self._n("A_log", "")].float()).contiguous()
        self.skip = tensors[self._n("D", "")].float().contiguous()
        self.norm_w = tensors[self._n("norm", "")].float().contiguous()
        self.w_o = tensors[self._n("o")]

    # A span longer than a piece is cut into pieces that run side by side (csrc/state_space.cu); a piece is a few chunks of
    # 64 tokens, as long as the step's tokens allow while the blocks still fill the multiprocessors.
    CHUNK = 64
    BLOCKS_PER_SM = 2

    def _on_tensor_cores(self, dtype) -> bool:
        G, N = self.groups, self.state_dim
        return dtype == torch.bfloat16 and ops.state_space_chunks_support(N, self.v_head_dim, self.channels, 0, self.inner,
                                                                          self.inner + G * N)

    @property
    def prepare_key(self):
        return ("state_space", self.num_heads, self.v_head_dim, self.state_dim, self.groups)

    def _pieces(self, ctx):
        """(item_span, item_c, span_first, num_items, chunk) for this step's spans, or None: token by token."""
        if ctx.decode_only or not self._on_tensor_cores(ctx.dtype):
            return None
        key = ("state_space_pieces", self.num_heads, self.v_head_dim, self.state_dim)
        hit = ctx.memo.get(key)
        if hit is not None:
            return hit
        chunk = 1 << 30
        longest = max(s.length for s in ctx.spans)
        if longest > 4 * self.CHUNK:
            blocks = self.num_heads * -(-self.v_head_dim // 64)             # of one piece
            wanted = max(1, L.num_sms(ctx.device) * self.BLOCKS_PER_SM // blocks)
            total = sum(s.length for s in ctx.spans)
            chunk = max(2 * self.CHUNK, -(-(-(-total // wanted)) // self.CHUNK) * self.CHUNK)
        counts = [-(-s.length // chunk) for s in ctx.spans]
        if max(counts) == 1:
            hit = (ctx.iota, ctx.zeros, ctx.iota, len(ctx.spans), 1 << 30)
        else:
            item_span = np.repeat(np.arange(len(counts), dtype=np.int32), counts)
            first = np.concatenate([[0], np.cumsum(counts)[:-1]]).astype(np.int32)
            item_c = (np.arange(len(item_span), dtype=np.int32) - first[item_span]).astype(np.int32)
            items = ctx.stage(np.stack([item_span, item_c]))
            hit = (items[0], items[1], ctx.stage(first), int(len(item_span)), int(chunk))
        ctx.shape_key.append(("state_space", hit[3], hit[4]))
        ctx.memo[key] = hit
        return hit

    def prepare(self, ctx, cache=None) -> None:
        self._pieces(ctx)

    def forward(self, x, residual, ctx, cache: CacheView) -> None:
        if isinstance(x, LazyNorm):
            x = x.materialize()
        if cache is None or cache.state is None or not cache.writes:
            raise ops.KernelError("state space: the run needs a state plane of its own (the recurrence advances it)")
        T = x.shape[0]
        H, G, N, vd, inner = self.num_heads, self.groups, self.state_dim, self.v_head_dim, self.inner
        fused = L.linear(x, self.w_in, None, L.STORE)               # [T, z | x | B | C | dt]
        spans = span_arrays(ctx)
        off, tail = cache.state_offset, cache.state_offset + self.state_floats
        xbc = torch.empty((T, self.channels), dtype=x.dtype, device=x.device)
        ops.conv_act(fused, inner, self.channels, self.w_conv, self.b_conv, "silu", spans, cache.state, tail, xbc,
                     fuse_tail=ctx.decode_only)
        if not ctx.decode_only and self.conv_taps > 1:
            ops.conv_tail_update(fused, inner, self.channels, self.conv_taps, spans, cache.state, tail)
        y = torch.empty((T, inner), dtype=torch.float32, device=x.device)
        dt0 = inner + self.channels
        ops.state_space(xbc, 0, inner, inner + G * N, fused[:, dt0: dt0 + H], self.dt_bias, self.rate, self.skip, spans, H, G, N,
                        vd, cache.state, off, y, single=ctx.decode_only, pieces=self._pieces(ctx))
        gated = torch.empty((T, inner), dtype=x.dtype, device=x.device)
        ops.gated_group_norm(y, fused[:, :inner], self.norm_w, self.norm_groups, self.norm_eps, gated)
        L.linear(gated, self.w_o, None, L.RESIDUAL, residual=residual)


register_part("mixer", "state_space", StateSpaceMixer)
