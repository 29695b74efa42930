"""A plain, slow evaluation of the Kutirax design: one function a mechanism, written from the design's equations in
float64 torch on the CPU.  It shares no code with the engine; the tests compare the engine with it.

``tensors`` maps checkpoint names to tensors; ``cfg`` is the config.json dictionary.  Every function takes whole
sequences (positions 0 .. T-1 of one request).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

F = torch.float64


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def stream_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The norm of the stream: its weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def token_shift(h: torch.Tensor, mix: torch.Tensor) -> torch.Tensor:
    """Every row moves towards the row before it (zeros before the first), channel by channel."""
    out = torch.empty_like(h)
    for t in range(h.shape[0]):
        before = h[t - 1] if t > 0 else torch.zeros_like(h[0])
        out[t] = h[t] + (before - h[t]) * mix
    return out


def rotate(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x ``[T, ..., >= dims]``: pairs (i, i + dims / 2) of the first ``dims`` dimensions turn by ``p * base^(-2i / dims)``."""
    y = x.clone()
    half = dims // 2
    for i in range(half):
        f = base ** (-2.0 * i / dims)
        a = torch.arange(x.shape[0], dtype=F) * f
        c, s = torch.cos(a), torch.sin(a)
        while c.dim() < x.dim() - 1:
            c, s = c.unsqueeze(-1), s.unsqueeze(-1)
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * c - v * s
        y[..., i + half] = v * c + u * s
    return y


def window_softmax(scores: torch.Tensor, window: Optional[int]) -> torch.Tensor:
    """scores ``[T, T]`` -> weights: row i sees the columns j with ``0 <= i - j < window``."""
    T = scores.shape[0]
    i = torch.arange(T)
    behind = i[:, None] - i[None, :]
    seen = (behind >= 0) if window is None else (behind >= 0) & (behind < window)
    return torch.softmax(scores.masked_fill(~seen, float("-inf")), dim=-1)


def latent_attention(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    """Keys and values are expanded head by head from the normed latent; nothing is folded."""
    T = h.shape[0]
    H, d, rd, vd, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    c_q = unit_rms(h @ t[f"{p}.dq"].T, eps) * t[f"{p}.dq.norm"]
    q = (c_q @ t[f"{p}.uq"].T).view(T, H, d + rd)
    down = h @ t[f"{p}.dkv"].T
    c = unit_rms(down[:, :r], eps) * t[f"{p}.dkv.norm"]
    k_rot = rotate(down[:, r:], rot["base"], rot["dims"])
    q_rot = rotate(q[..., d:], rot["base"], rot["dims"])
    k = (c @ t[f"{p}.uk"].T).view(T, H, d)
    v = (c @ t[f"{p}.uv"].T).view(T, H, vd)
    window = m["mask"]["size"] if m.get("mask") else None
    out = torch.zeros(T, H, vd, dtype=h.dtype)
    for n in range(H):
        scores = (q[:, n, :d] @ k[:, n].T + q_rot[:, n] @ k_rot.T) * m["scale"]
        out[:, n] = window_softmax(scores, window) @ v[:, n]
    return out.reshape(T, H * vd) @ t[f"{p}.o"].T


def causal_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """``y[t, c] = b[c] + sum_j w[c, j] u[t - taps + 1 + j, c]``, zeros before the first token."""
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        y[t] = b
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] = y[t] + w[:, j] * u[s]
    return y


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def state_space(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, A_log: torch.Tensor,
                D: torch.Tensor) -> torch.Tensor:
    """The recurrence token by token.  x ``[T, H, vdim]``, B and C ``[T, G, N]``, dt ``[T, H]`` (after the softplus)."""
    T, H, vd = x.shape
    G, N = B.shape[1], B.shape[2]
    S = torch.zeros(H, N, vd, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """``y * silu(z)``, then each of ``parts`` equal parts by its own root mean square, then the weight."""
    T, n = y.shape
    return unit_rms((y * silu(z)).view(T, parts, n // parts), eps).reshape(T, n) * w


def mamba2(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, vd, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    z, xbc, dt = (h @ t[f"{p}.in"].T).split([inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(causal_conv(xbc, t[f"{p}.conv"], t[f"{p}.conv.b"]))
    x, B, C = xbc.split([inner, G * N, G * N], dim=-1)
    dt = torch.nn.functional.softplus(dt + t[f"{p}.dt_bias"], threshold=200.0)
    y = state_space(x.reshape(T, H, vd), B.reshape(T, G, N), C.reshape(T, G, N), dt, t[f"{p}.A_log"], t[f"{p}.D"])
    return gated_group_norm(y.reshape(T, inner), z, t[f"{p}.norm"], m["norm_groups"], eps) @ t[f"{p}.o"].T


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2}


def squared_relu_mlp(h: torch.Tensor, t: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return torch.clamp(h @ t[f"{p}.up"].T, min=0.0) ** 2 @ t[f"{p}.down"].T


def route(h: torch.Tensor, w: torch.Tensor, b: torch.Tensor, top: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """(ids ``[T, top]``, weights ``[T, top]``): the largest logits and the softmax over them alone."""
    z = h @ w.T + b
    values, ids = torch.topk(z, top, dim=-1)
    return ids, torch.softmax(values, dim=-1)


def experts(h: torch.Tensor, mlp: dict, t: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    ids, weights = route(h, t[f"{p}.router"], t[f"{p}.router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for i in range(h.shape[0]):
        for e, w in zip(ids[i].tolist(), weights[i]):
            a = silu(t[f"{p}.e{e}.gate"] @ h[i]) * (t[f"{p}.e{e}.up"] @ h[i])
            out[i] += w * (t[f"{p}.e{e}.down"] @ a)
    return out


def feed_forward(h: torch.Tensor, mlp: dict, t: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return squared_relu_mlp(h, t, p) if mlp["kind"] == "dense" else experts(h, mlp, t, p)


def layer(x: torch.Tensor, i: int, spec: dict, t: Dict[str, torch.Tensor], eps: float, m: float) -> torch.Tensor:
    h = token_shift(stream_norm(x, t[f"l{i}.norm1"], eps), t[f"l{i}.shift"])
    branches = MIXERS[spec["type"]](h, spec["mixer"], t, f"l{i}.mix", eps)
    if spec.get("mlp") is not None:
        branches = branches + feed_forward(stream_norm(x, t[f"l{i}.norm2"], eps), spec["mlp"], t, f"l{i}.mlp")
    return x + m * branches


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens: List[int],
            layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence."""
    t = {k: v.to(F) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])
    x = t["embed"][torch.tensor(tokens, dtype=torch.long)]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, i, spec, t, eps, float(cfg.get("residual_mult", 1.0)))
        if layers_out is not None:
            layers_out.append(x.clone())
    return stream_norm(x, t["final.norm"], eps) @ t["embed"].T
