"""Tiny Laralix configurations for the tests, and random weights for them drawn here (names and shapes restated from the
design, not taken from the engine).  The configurations differ in every size, in the order of the layers, in where the loop lies,
in which values happen to be equal, 1 or absent, and in which kernels the engine picks for them."""
import copy
import json
import os
from typing import Dict, Optional

import torch


def _parallel(heads, kv, dim, vdim, size, cap, rheads, rkv, rdim, rvdim, conv, scale=None):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5}
    if cap is not None:
        left["softcap"] = cap
    if size is not None:
        left["mask"] = {"size": size}
    right = {"heads": rheads, "kv_heads": rkv, "dim": rdim, "vdim": rvdim, "conv": conv}
    return {"type": "parallel", "mixer": {"left": left, "right": right}}


def _parallel_2(heads, kv, dim, size, keep, rheads, rdim, rvdim, tau, rank, ls, rs, scale=None):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5}
    if size is not None:
        left["mask"] = {"size": size, "keep_first": keep}
    return {"type": "parallel_2", "mixer": {"left": left, "left_scale": ls, "right_scale": rs,
                                            "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "tau": tau, "decay_rank": rank}}}


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base=10000.0, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
            "kv_rank": kv_rank, "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}}


def _ff(layer, ff: Optional[int] = None):
    return dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def _model(vocab, width, eps, emb, logit, layers, loop=None):
    cfg = {"architecture": "Laralix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": emb},
           "logit_scale": logit, "layers": layers}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: odd sizes everywhere (CUDA-core kernels in both precisions), values narrower and wider than keys, windows shorter and longer
# than a page, kept tokens that end inside a page, a layer without feed-forward, the loop in the middle.
LAR_A = _model(303, 44, 1e-5, 5.0, 0.7, [
    _ff(_parallel(6, 3, 10, 14, 9, 8.0, 4, 2, 6, 10, 3), 20),
    _ff(_parallel_2(4, 2, 12, 11, 3, 3, 10, 7, 5.0, 3, 0.8, 1.3), 28),
    _ff(_latent(3, 10, 6, 14, 18, 22, base=500.0)),
    _ff(_parallel(3, 3, 9, 7, 40, 15.0, 2, 1, 11, 5, 5), 17),
], loop=(1, 3, 2))
# B: sizes of the tensor-core kernels in bfloat16: heads of 64 and 128, windows across tiles, kept tokens beyond a page and a
# stretch of more than a tile of 128; the loop at the start, three times.
LAR_B = _model(517, 128, 1e-6, 9.0, 1.5, [
    _ff(_parallel(4, 1, 64, 64, 150, 12.0, 2, 2, 32, 64, 4), 96),
    _ff(_parallel_2(8, 2, 64, 130, 20, 4, 16, 32, 12.0, 16, 1.1, 0.6), 192),
    _ff(_latent(6, 32, 16, 48, 64, 96, base=50000.0), 64),
    _ff(_parallel_2(2, 2, 128, 16, 140, 1, 96, 40, 3.0, 8, 0.9, -0.7), 72),
    _ff(_parallel(3, 3, 128, 128, 33, None, 3, 1, 64, 16, 2), 80),
], loop=(0, 3, 3))
# C: what the others make unequal is equal, 1 or absent here: one head, a window of one token with none and with one kept, no
# mask, no cap, one tap, tau 1, rank 1, a loop of one pass over every layer, scales of 1.
LAR_C = _model(97, 32, 1e-6, 1.0, 1.0, [
    _ff(_parallel(1, 1, 8, 8, 1, None, 1, 1, 8, 8, 1), 8),
    _ff(_parallel_2(1, 1, 8, 1, 0, 1, 8, 8, 1.0, 1, 1.0, 1.0), 8),
    _ff(_parallel_2(2, 1, 16, 1, 1, 2, 4, 16, 1.0, 2, 0.0, 1.0)),
    _ff(_parallel_2(2, 2, 8, None, 0, 1, 8, 4, 2.0, 2, 1.0, 1.0), 16),
    _ff(_parallel(2, 1, 8, 8, None, 3.0, 2, 1, 4, 12, 2), 8),
    _ff(_latent(1, 8, 8, 8, 8, 8, scale=1.0), 8),
], loop=(0, 6, 1))
# D: no loop; many heads (slopes close together), wide groups, more than one thread a column in the recurrences (heads of 72 and
# 130), eight taps, windows and kept tokens of whole pages.
LAR_D = _model(211, 50, 1e-5, 3.0, 2.5, [
    _ff(_latent(17, 6, 8, 10, 12, 40, base=100.0), 30),
    _ff(_parallel(20, 4, 6, 12, 16, 30.0, 6, 2, 72, 9, 8), 24),
    _ff(_parallel_2(18, 1, 10, 32, 16, 2, 130, 12, 16.0, 20, 1.4, 0.5)),
])
# E: one latent layer wide enough for the CUDA-core kernel's shared heads; head groups of 16 over keys of 64; the loop at the end.
LAR_E = _model(150, 64, 1e-6, 2.0, 0.5, [
    _ff(_parallel_2(16, 1, 64, 64, 5, 3, 24, 16, 8.0, 4, 0.7, 0.7), 40),
    _ff(_latent(5, 24, 64, 16, 32, 512, base=1000.0), 40),
    _ff(_parallel(16, 1, 64, 64, 100, 20.0, 2, 2, 16, 72, 3), 48),
], loop=(1, 3, 4))
CONFIGS = {"A": LAR_A, "B": LAR_B, "C": LAR_C, "D": LAR_D, "E": LAR_E}
PAGE_SIZE = {"A": 16, "B": 16, "C": 8, "D": 16, "E": 32}


def config(name):
    return copy.deepcopy(CONFIGS[name])


def random_config(rng, tensor_core: bool):
    """A configuration drawn at random: two to five layers of any kind and size (with ``tensor_core`` heads of 64 and 128 and
    multiples of eight), windows from 1 to 200 or none, any loop or none."""
    width = rng.choice([64, 96, 192]) if tensor_core else rng.choice([40, 57, 72, 100])
    pick = (lambda lo, hi: 8 * rng.randint(max(1, lo // 8), hi // 8)) if tensor_core else rng.randint
    windows = [None, 1, 2, 7, 16, 17, 31, 64, 100, 129, 200]
    layers = []
    for _ in range(rng.randint(2, 5)):
        kind = rng.choice(["p", "p", "q", "q", "l"])
        G = rng.choice([1, 2, 3])
        H = G * rng.randint(1, 5)
        dim = rng.choice([64, 128]) if tensor_core else rng.randint(5, 40)
        if kind == "p":
            RG = rng.choice([1, 2])
            layer = _parallel(H, G, dim, dim if tensor_core and rng.random() < 0.7 else rng.randint(4, 40), rng.choice(windows),
                              rng.choice([None, 5.0, 30.0]), RG * rng.randint(1, 3), RG, pick(5, 72), pick(4, 72), rng.randint(1, 6))
        elif kind == "q":
            layer = _parallel_2(H, G, dim, rng.choice(windows), rng.choice([0, 1, 3, 4, 16, 19, 70]), rng.randint(1, 4), pick(4, 72),
                                pick(4, 72), rng.choice([1.0, 4.0, 16.0, 30.0]), pick(2, 24), rng.choice([1.0, 0.6, -1.2]),
                                rng.choice([1.0, 0.4, 1.3]))
        else:
            layer = _latent(rng.randint(1, 12), pick(4, 40), pick(8, 24) if tensor_core else 2 * rng.randint(1, 12), pick(4, 40),
                            pick(4, 64), pick(4, 130), base=rng.choice([100.0, 10000.0, 1000000.0]))
        layers.append(_ff(layer, None if rng.random() < 0.2 else pick(6, 96)))
    loop = None
    if rng.random() < 0.7:
        a = rng.randrange(len(layers))
        loop = (a, rng.randint(a + 1, len(layers)), rng.randint(1, 3))
    return _model(rng.choice([97, 301, 523]), width, rng.choice([1e-6, 1e-5]), rng.choice([1.0, 4.0, 12.0]), rng.choice([1.0, 0.5, 3.0]),
                  layers, loop)


def tensor_shapes(cfg) -> Dict[str, tuple]:
    """Every tensor of a model of this design, by the naming rule of its checkpoints."""
    D, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, D), "head": (V, D), "final.norm": (D,)}
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], D)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", layer["mixer"]
        out[f"l{i}.norm1"] = (D,)
        if layer["type"] == "latent_attention":
            H, d, rd, vd, qr, r = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            out.update({f"{p}.dq": (qr, D), f"{p}.dq.norm": (qr,), f"{p}.uq": (H * (d + rd), qr), f"{p}.dkv": (r + rd, D),
                        f"{p}.dkv.norm": (r,), f"{p}.uk": (H * d, r), f"{p}.uv": (H * vd, r), f"{p}.o": (D, H * vd)})
        else:
            a, b, l, r = m["left"], m["right"], f"{p}.left", f"{p}.right"
            H, G, d, vd = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            out.update({f"{l}.q": (H * d, D), f"{l}.k": (G * d, D), f"{l}.o": (D, H * vd)})
            h, e, ve = b["heads"], b["dim"], b["vdim"]
            out.update({f"{r}.v": (h * ve, D), f"{r}.g": (h * ve, D), f"{r}.norm": (ve,), f"{r}.o": (D, h * ve)})
            if layer["type"] == "parallel":
                g, n = b["kv_heads"], b["conv"]
                out.update({f"{l}.v": (G * vd, D), f"{l}.q.norm": (d,), f"{l}.k.norm": (d,), f"{l}.out": (D,), f"{r}.out": (D,),
                            f"{r}.q": (g * e, D), f"{r}.k": (g * e, D), f"{r}.q.conv": (g * e, n), f"{r}.k.conv": (g * e, n),
                            f"{r}.v.conv": (h * ve, n), f"{r}.b": (h, D), f"{r}.a": (h, D), f"{r}.A_log": (h,), f"{r}.dt_bias": (h,)})
            else:
                out.update({f"{l}.q.norm": (H * d,), f"{l}.k.norm": (G * d,), f"{r}.q": (h * e, D), f"{r}.k": (h * e, D),
                            f"{r}.a1": (b["decay_rank"], D), f"{r}.a2": (h * e, b["decay_rank"]), f"{r}.a2.b": (h * e,)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.norm2": (D,), f"l{i}.mlp.gate": (ff, D), f"l{i}.mlp.up": (ff, D), f"l{i}.mlp.down": (D, ff)})
    return out


def random_weights(cfg, seed: int, store=torch.float32) -> Dict[str, torch.Tensor]:
    """Weights that keep activations of order one: matrices N(0, 1/in), norm weights around zero where the design adds 1 and
    around one elsewhere, decays that forget within a few to a few hundred tokens.  Rounded once to ``store``."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        tail = name.split(".")[-1]
        rn = torch.randn(shape, generator=g)
        if tail in ("norm1", "norm2") or name == "final.norm":
            t = 0.1 * rn
        elif tail in ("norm", "out"):
            t = 1.0 + 0.2 * rn
        elif tail == "dt_bias":
            t = -2.0 + rn
        elif tail == "A_log":
            t = -0.5 + rn
        elif tail == "conv":
            t = 0.5 * rn
        elif tail == "step":
            t = 0.5 * rn
        elif name.endswith("a2.b"):
            t = 1.0 + rn
        elif name == "embed":
            t = rn
        else:
            t = rn / shape[1] ** 0.5
        out[name] = t.to(store).contiguous()
    return out


def write_model(cfg, weights, out_dir: str, ranks_in_config: bool = False) -> str:
    """A folder as checkpoints of the design come: the decays' ranks are in the tensors' shapes alone, unless asked otherwise."""
    from lightllm_b200.weights import save_file
    os.makedirs(out_dir, exist_ok=True)
    cfg = copy.deepcopy(cfg)
    if not ranks_in_config:
        for layer in cfg["layers"]:
            layer["mixer"].get("right", {}).pop("decay_rank", None)
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(weights, os.path.join(out_dir, "model.safetensors"))
    return out_dir
