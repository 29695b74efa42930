"""A plain, slow evaluation of the Laralix design: one function a mechanism, written from the design's equations in float64
torch on the CPU.  It shares no code with the engine; the tests compare the engine with it.

``tensors`` maps checkpoint names to tensors; ``cfg`` is the config.json dictionary.  Every function takes whole sequences
(positions 0 .. T-1 of one request).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F = torch.float64


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def layer_norm1p(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The norm around a layer's branches and before the head: its weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x / (1.0 + torch.exp(-x))


def short_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``y[t, c] = sum_j w[c, j] * u[t - taps + 1 + j, c]`` with zeros before the first token."""
    T, C = u.shape
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def visible(i: int, j: int, size: Optional[int], keep: int = 0) -> bool:
    return j <= i and (size is None or i - j < size or j < keep)


def slopes(heads: int) -> List[float]:
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def attention(q, k, v, scale: float, size: Optional[int] = None, keep: int = 0, softcap: Optional[float] = None,
              distance: bool = False, plus_one: bool = False, start: int = 0) -> torch.Tensor:
    """q ``[T, H, dim]`` (row i at position start + i), k ``[.., G, dim]``, v ``[.., G, vdim]``; see :func:`visible` for the mask.  ``distance``: the bias of a
    head's slope times the distance is taken off the (capped) score; ``plus_one``: one more in the denominator."""
    T, H, _ = q.shape
    kv = torch.arange(H) // (H // k.shape[1])                                  # the kv head of every query head
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    slope = torch.tensor(slopes(H), dtype=q.dtype)
    for row in range(T):
        i = start + row
        js = torch.tensor([j for j in range(i + 1) if visible(i, j, size, keep)])
        s = torch.einsum("hd,jhd->hj", q[row], k[js][:, kv]) * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        if distance:
            s = s - slope[:, None] * (i - js).to(q.dtype)
        m = s.max(-1, keepdim=True).values
        if plus_one:
            m = torch.clamp(m, min=0.0)
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True) + (torch.exp(-m) if plus_one else 0.0)
        out[row] = torch.einsum("hj,jhe->he", e / den, v[js][:, kv])
    return out


def distance_attention(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    """The left side of 'parallel'."""
    T, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ W[f"{p}.q"].T).view(T, H, d), W[f"{p}.q.norm"], eps)
    k = rms_norm((h @ W[f"{p}.k"].T).view(T, G, d), W[f"{p}.k.norm"], eps)
    v = (h @ W[f"{p}.v"].T).view(T, G, vd)
    o = attention(q, k, v, float(m["scale"]), (m.get("mask") or {}).get("size"), 0, m.get("softcap"), True, True)
    return o.reshape(T, H * vd) @ W[f"{p}.o"].T


def delta_rule(q, k, v, g, beta) -> torch.Tensor:
    """One head.  q, k ``[T, dim]``, v ``[T, vdim]``, g and beta ``[T]``; the state ``[dim, vdim]`` starts at zero."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def unit_vector(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(h, W, p: str) -> torch.Tensor:
    """g ``[T, heads]``."""
    z = h @ W[f"{p}.a"].T + W[f"{p}.dt_bias"]
    return torch.exp(-torch.exp(W[f"{p}.A_log"]) * torch.logaddexp(z, torch.zeros_like(z)))


def head_delta(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    """The right side of 'parallel'."""
    T, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def proj(n):
        y = h @ W[f"{p}.{n}"].T
        return silu(short_conv(y, W[f"{p}.{n}.conv"]))
    q = unit_vector(proj("q").view(T, G, d)) * d ** -0.5
    k = unit_vector(proj("k").view(T, G, d))
    v = proj("v").view(T, H, vd)
    beta = torch.sigmoid(h @ W[f"{p}.b"].T)
    g = head_decay(h, W, p)
    o = torch.stack([delta_rule(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], g[:, i], beta[:, i]) for i in range(H)], 1)
    o = unit_rms(o, eps) * W[f"{p}.norm"] * silu(h @ W[f"{p}.g"].T).view(T, H, vd)
    return o.reshape(T, H * vd) @ W[f"{p}.o"].T


def parallel(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    a = rms_norm(distance_attention(h, W, f"{p}.left", m["left"], eps), W[f"{p}.left.out"], eps)
    b = rms_norm(head_delta(h, W, f"{p}.right", m["right"], eps), W[f"{p}.right.out"], eps)
    return 0.5 * (a + b)


def kept_first_attention(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    """The left side of 'parallel_2'."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rms_norm(h @ W[f"{p}.q"].T, W[f"{p}.q.norm"], eps).view(T, H, d)
    k0 = h @ W[f"{p}.k"].T
    k = rms_norm(k0, W[f"{p}.k.norm"], eps).view(T, G, d)
    mask = m.get("mask") or {}
    o = attention(q, k, k0.view(T, G, d), float(m["scale"]), mask.get("size"), mask.get("keep_first", 0))
    return o.reshape(T, H * d) @ W[f"{p}.o"].T


def gated_linear(q, k, v, alpha) -> torch.Tensor:
    """One head.  q, k, alpha ``[T, dim]``, v ``[T, vdim]``."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def channel_decay(h, W, p: str, tau: float) -> torch.Tensor:
    z = (h @ W[f"{p}.a1"].T) @ W[f"{p}.a2"].T + W[f"{p}.a2.b"]
    return torch.sigmoid(z) ** (1.0 / tau)


def gated_linear_attention(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    """The right side of 'parallel_2'."""
    T, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W[f"{p}.q"].T).view(T, H, d) * d ** -0.5
    k = (h @ W[f"{p}.k"].T).view(T, H, d)
    v = (h @ W[f"{p}.v"].T).view(T, H, vd)
    alpha = channel_decay(h, W, p, float(m["tau"])).view(T, H, d)
    o = torch.stack([gated_linear(q[:, i], k[:, i], v[:, i], alpha[:, i]) for i in range(H)], 1)
    o = rms_norm(o, W[f"{p}.norm"], eps).reshape(T, H * vd)
    return (o * silu(h @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T


def parallel_2(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    return (float(m["left_scale"]) * kept_first_attention(h, W, f"{p}.left", m["left"], eps)
            + float(m["right_scale"]) * gated_linear_attention(h, W, f"{p}.right", m["right"], eps))


def rotate_pairs(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x ``[T, heads, n]``, position t in row t: dimensions 2i and 2i + 1 of the first ``dims`` turn together."""
    dims, base = rot["dims"], float(rot["base"])
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = t * base ** (-2.0 * i / dims)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            out[t, :, 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[t, :, 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def latent_attention(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d, rd, vd, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ W[f"{p}.dq"].T, W[f"{p}.dq.norm"], eps)
    q = (cq @ W[f"{p}.uq"].T).view(T, H, d + rd)
    down = h @ W[f"{p}.dkv"].T
    c = rms_norm(down[:, :r], W[f"{p}.dkv.norm"], eps)
    kr = rotate_pairs(down[:, None, r:], m["rot"]).expand(T, H, rd)
    q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], m["rot"])], dim=-1)
    k = torch.cat([(c @ W[f"{p}.uk"].T).view(T, H, d), kr], dim=-1)
    v = (c @ W[f"{p}.uv"].T).view(T, H, vd)
    o = attention(q, k, v, float(m["scale"]), (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * vd) @ W[f"{p}.o"].T


def dense(h, W, p: str) -> torch.Tensor:
    return (silu(h @ W[f"{p}.gate"].T) * (h @ W[f"{p}.up"].T)) @ W[f"{p}.down"].T


MIXERS = {"parallel": parallel, "parallel_2": parallel_2, "latent_attention": latent_attention}


def run_list(cfg: dict) -> List[Tuple[int, Optional[int]]]:
    """(layer, pass number if the layer opens a pass of the loop else None) in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        for i in range(loop["start"], loop["stop"]):
            out.append((i, t if i == loop["start"] else None))
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(tokens, cfg: dict, tensors: Dict[str, torch.Tensor], dtype=F):
    """Logits ``[T, vocab]`` of one whole sequence, and the stream after every run of a layer."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    x0 = x.clone()
    streams = []
    for i, opens in run_list(cfg):
        if opens is not None:
            if opens > 0:
                x = x + x0
            x = x + W["loop.step"][opens]
        layer, p = cfg["layers"][i], f"l{i}"
        x = x + MIXERS[layer["type"]](layer_norm1p(x, W[f"{p}.norm1"], eps), W, f"{p}.mix", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + dense(layer_norm1p(x, W[f"{p}.norm2"], eps), W, f"{p}.mlp")
        streams.append(x.clone())
    logits = layer_norm1p(x, W["final.norm"], eps) @ W["head"].T * float(cfg["logit_scale"])
    return logits, torch.stack(streams)
