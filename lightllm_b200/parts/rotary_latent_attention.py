"""Attention over a cached low-rank latent with a rotated key part shared by all heads and queries through a latent of
their own."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..config import PartSpec, register_part
from ..csrc import ops
from ..weights import WeightSpec
from . import linear as L
from .attention import AttentionMixer
from .base import CacheView, LazyNorm


class RotaryLatentAttentionMixer(AttentionMixer):
    """Latent attention with decoupled rotary positions::

        c_q = rms(W_dq x) * g_q;   q_h = W_uq,h c_q = [q'_h (head_dim) | q''_h (rot_dim)]
        [c | k''] = W_dkv x;       c <- rms(c) * g_c (``rank`` numbers);   q''_h, k'' <- rotated by position
        s = scale (q'_h . W_uk,h c + q''_h . k'');   o_h = W_uv,h sum p c;   out = W_o [o_1 .. o_H]

    The cache keeps ``[c | k'']`` a token and nothing else (one kv head of ``rank + rot_dim``, no value rows).  The key
    up-projection is applied to the query, ``q'.W_uk c = (W_uk^T q').c``, and the value up-projection to the mixed latents, so
    the kernels see multi-query attention over the cached rows whose first ``rank`` numbers are the values, and nothing of
    the context is ever expanded.

    ``window``: a query sees the latest ``window`` keys (itself included).  In bfloat16 the attention runs on the kernels of
    csrc/latent_attention_tcgen05.cu (steps with portions of prompts) and csrc/latent_attention.cu (single tokens, latents wider
    than 256), otherwise (float32, widths that are no multiples of 8) on the CUDA-core attention kernels.  Norms, angles, scores and
    the softmax are float32 in both precisions."""

    graph_safe = True
    accepts_lazy_norm = False

    def __init__(self, prefix: str, hidden_size: int, num_heads: int, head_dim: int, rot_dim: int, v_head_dim: int, q_rank: int,
                 rank: int, position: Optional[PartSpec] = None, norm_eps: float = 1e-6, scale: Optional[float] = None,
                 window: Optional[int] = None, names: Optional[Dict[str, str]] = None, weight_suffix: str = ".weight",
                 norm_ending: str = "norm"):
        base = {"dq": "q_down", "uq": "q_up", "dkv": "kv_down", "uk": "k_up", "uv": "v_up", "o": "o_proj"}
        base.update(names or {})
        # the attention kernels' geometry: one kv head of rank + rot_dim whose first `rank` numbers are the values
        super().__init__(prefix, hidden_size, num_heads, 1, rank + rot_dim, position=position, qkv_bias=False, out_bias=False,
                         window=window, scale=scale if scale is not None else (head_dim + rot_dim) ** -0.5, names=base,
                         weight_suffix=weight_suffix, v_head_dim=rank)
        self.values_in_keys = True
        self.q_dim, self.rot_dim, self.out_dim = int(head_dim), int(rot_dim), int(v_head_dim)
        self.q_rank, self.rank, self.norm_eps, self.norm_ending = int(q_rank), int(rank), float(norm_eps), norm_ending
        table = self.position.rotary_table()
        if rot_dim and (table is None or table[1] != rot_dim):
            raise ValueError(f"the shared key part of {rot_dim} is rotated whole; the position encoding rotates "
                             f"{0 if table is None else table[1]}")
        self.w_down = self.w_uq = self.w_q_up = self.w_v_up = self.q_norm_w = self.c_norm_w = None

    def weight_specs(self) -> List[WeightSpec]:
        D, H, r = self.hidden_size, self.num_heads, self.rank
        return [WeightSpec(self._n("dq", "weight"), (self.q_rank, D)),
                WeightSpec(self._n("dq", self.norm_ending), (self.q_rank,), init=("one_plus_normal", 0.1)),
                WeightSpec(self._n("uq", "weight"), (H * (self.q_dim + self.rot_dim), self.q_rank)),
                WeightSpec(self._n("dkv", "weight"), (r + self.rot_dim, D)),
                WeightSpec(self._n("dkv", self.norm_ending), (r,), init=("one_plus_normal", 0.1)),
                WeightSpec(self._n("uk", "weight"), (H * self.q_dim, r)),
                WeightSpec(self._n("uv", "weight"), (H * self.out_dim, r)),
                WeightSpec(self._n("o", "weight"), (D, H * self.out_dim))] + self.position.weight_specs()

    def bind(self, tensors, dtype, device) -> None:
        H, r = self.num_heads, self.rank
        dq, dkv = tensors[self._n("dq", "weight")], tensors[self._n("dkv", "weight")]
        wdt = torch.float32 if torch.float32 in (dq.dtype, dkv.dtype) else dq.dtype
        ws = [dq.to(wdt), dkv.to(wdt)]
        pad = -(self.q_rank + r + self.rot_dim) % 8          # whole 16-byte pieces a row of the projection's output
        if pad:
            ws.append(torch.zeros((pad, self.hidden_size), dtype=wdt, device=dq.device))
        self.w_down = torch.cat(ws, dim=0).contiguous()
        self.w_uq = tensors[self._n("uq", "weight")]
        # [H, rank, dim]: row o of head h is column o of that head's key up-projection; the per-head contraction takes its
        # weights in the activations' dtype (also where a checkpoint stores them in 32 bits)
        self.w_q_up = tensors[self._n("uk", "weight")].view(H, self.q_dim, r).to(dtype).transpose(1, 2).contiguous()
        self.w_v_up = tensors[self._n("uv", "weight")].view(H, self.out_dim, r).to(dtype).contiguous()
        self.w_o = tensors[self._n("o", "weight")]
        self.q_norm_w = tensors[self._n("dq", self.norm_ending)].float().contiguous()
        self.c_norm_w = tensors[self._n("dkv", self.norm_ending)].float().contiguous()
        self.position.bind(tensors, dtype, device)

    # ------------------------------------------------------------------------------------------
    def _on_tensor_cores(self, dtype) -> bool:
        return dtype == torch.bfloat16 and ops.latent_attention_supports(self.head_dim, self.rank)

    def prepare(self, ctx, cache=None) -> None:
        if not self._on_tensor_cores(ctx.dtype):
            super().prepare(ctx, cache)

    def _key_pieces(self, ctx) -> int:
        """Pieces that the keys of single tokens are cut into: enough blocks for the multiprocessors, at least two tiles of
        64 keys each (a function of what a CUDA graph's key holds)."""
        if not ctx.decode_only:
            return 1
        bound = ctx.max_pages * ctx.page_size
        window = self.kernel_window()
        span = bound if window == 0 else min(bound, abs(window))
        blocks = ctx.num_spans * -(-self.num_heads // 64)
        return max(1, min(ops.LATENT_MAX_SPLITS, 2 * L.num_sms(ctx.device) // blocks, span // 128))

    def forward(self, x, residual, ctx, cache: CacheView) -> None:
        if isinstance(x, LazyNorm):
            x = x.materialize()
        T = x.shape[0]
        H, r, rd, d, W = self.num_heads, self.rank, self.rot_dim, self.q_dim, self.head_dim
        table = self.position.rotary_table() or (None, 0, False)
        inv_freq, _, interleaved = table
        down = L.linear(x, self.w_down, None, L.STORE)              # [T, query latent | latent | rotated part]
        c_q = torch.empty((T, self.q_rank), dtype=x.dtype, device=x.device)
        ops.latent_prepare(down, 0, self.q_rank, self.q_rank + r, self.q_rank, r, rd, self.q_norm_w, self.c_norm_w, inv_freq,
                           interleaved, ctx.positions, ctx.slot_mapping[cache.group] if cache.writes else None, c_q,
                           cache.k if cache.writes else None, self.norm_eps)
        heads = L.linear(c_q, self.w_uq, None, L.STORE)             # [T, H * (dim | rot_dim)]
        q = torch.empty((T, H * W), dtype=x.dtype, device=x.device)
        ops.head_linear(heads, 0, self.w_q_up, q, x_head=d + rd, out_head=W,
                        rotate=(d, r, rd, ctx.positions, inv_freq, interleaved) if rd else None)
        mixed = torch.empty((T, H * r), dtype=x.dtype, device=x.device)
        self.attend(q, cache, ctx, mixed)                           # sum_j p_ij c_j
        out = torch.empty((T, H * self.out_dim), dtype=x.dtype, device=x.device)
        ops.head_linear(mixed, 0, self.w_v_up, out)
        L.linear(out, self.w_o, None, L.RESIDUAL, residual=residual)

    def attend(self, q, cache: CacheView, ctx, out) -> None:
        if not self._on_tensor_cores(q.dtype):
            super().attend(q, cache, ctx, out)
            return
        if not ctx.decode_only and ops.latent_attention_tcgen05_supports(self.head_dim, self.rank, ctx.page_size):
            ops.latent_attention_tcgen05(q, cache.k, out, ctx.span_row, ctx.span_len, ctx.span_pos, ctx.num_spans,
                                         ctx.block_tables[cache.group], ctx.max_pages, ctx.page_size, self.num_heads, self.head_dim,
                                         self.rank, self.kernel_window(), self.scale, sinks=self.sinks)
            return
        ops.latent_attention(q, cache.k, out, ctx.span_row, ctx.span_len, ctx.span_pos, ctx.num_spans, ctx.block_tables[cache.group],
                             ctx.max_pages, ctx.page_size, self.num_heads, self.head_dim, self.rank, self.kernel_window(),
                             self.scale, ctx.decode_only, self._key_pieces(ctx), sinks=self.sinks)


register_part("mixer", "rotary_latent_attention", RotaryLatentAttentionMixer)
