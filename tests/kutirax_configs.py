"""Tiny Kutirax configurations for the tests, and random weights for them drawn here (names and shapes restated from the
design, not taken from the engine).  The configurations differ in every size, in the order of the layers, in which values
happen to be equal, 1 or absent, and in which kernels the engine picks for them."""
import copy
import json
import os
from typing import Dict

import torch


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, base=10000.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m}


def _mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def _ff(layer, ff=None, experts=None, top=None):
    layer = dict(layer)
    if ff is None:
        layer["mlp"] = None
    elif experts is None:
        layer["mlp"] = {"kind": "dense", "ff": ff}
    else:
        layer["mlp"] = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return layer


def _model(vocab, width, eps, mult, layers):
    cfg = {"architecture": "Kutirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if mult is not None:
        cfg["residual_mult"] = mult
    return cfg


# A: odd sizes everywhere (CUDA-core kernels in both precisions); windows shorter and longer than a page; a layer without
# feed-forward; three norm groups over four heads.
KUT_A = _model(301, 44, 1e-5, 0.7, [
    _ff(_mamba(3, 10, 6, 1, 3, 1), 20),
    _ff(_latent(3, 10, 6, 14, 18, 22, 9, base=500.0), 12, 5, 2),
    _ff(_mamba(4, 6, 10, 2, 4, 3)),
    _ff(_latent(2, 7, 2, 5, 9, 13, 33), 10, 3, 1),
])
# B: sizes of the tensor-core kernels in bfloat16: latents of 96 and 256, states of 64 and 128 in one and two groups, windows
# across tiles and pages, eight experts (grouped contractions from 48 rows on, pair by pair for few rows).
KUT_B = _model(517, 128, 1e-6, 0.35, [
    _ff(_mamba(4, 32, 64, 2, 4, 4), 64, 8, 2),
    _ff(_latent(6, 32, 16, 48, 64, 96, 150, base=50000.0), 256),
    _ff(_mamba(2, 64, 128, 1, 2, 1), 192),
    _ff(_latent(3, 64, 32, 32, 40, 256, 70), 32, 6, 3),
])
# C: what the others make unequal is equal, 1 or absent here: one head, a window of one token and a layer without a mask, one
# tap (no convolution over time), no residual multiplier, every expert chosen, one expert of which one is chosen.
KUT_C = _model(97, 32, 1e-6, None, [
    _ff(_mamba(1, 8, 8, 1, 1, 1), 8, 2, 2),
    _ff(_latent(1, 8, 8, 8, 8, 8, 1, scale=1.0), 16, 1, 1),
    _ff(_latent(2, 8, 8, 8, 16, 16, None), 8),
    _ff(_mamba(2, 8, 8, 2, 2, 2)),
])
# D: many heads (more pairs of token and head than a tile holds), key rows that are no multiple of eight numbers, a state wider
# than the chunk kernels' rows allow, five taps, eight norm groups, a window of whole pages.
KUT_D = _model(211, 50, 1e-5, 1.3, [
    _ff(_latent(20, 6, 4, 8, 30, 24, 16, base=100.0), 24, 4, 3),
    _ff(_mamba(8, 4, 130, 4, 5, 8), 24, 2, 1),
    _ff(_latent(17, 6, 8, 10, 12, 40, 48), 30),
])
# E: a latent of 512 (too wide for the tensor memory's kernel), a state of 256 with value rows of 72, a state of 24.
KUT_E = _model(150, 64, 1e-6, 0.6, [
    _ff(_latent(5, 24, 64, 16, 32, 512, 100, base=1000.0), 40),
    _ff(_mamba(2, 72, 256, 1, 4, 2), 16, 7, 2),
    _ff(_mamba(3, 16, 24, 3, 3, 1), 48),
])
CONFIGS = {"A": KUT_A, "B": KUT_B, "C": KUT_C, "D": KUT_D, "E": KUT_E}
PAGE_SIZE = {"A": 16, "B": 16, "C": 8, "D": 16, "E": 32}


def config(name):
    return copy.deepcopy(CONFIGS[name])


def random_config(rng, tensor_core: bool):
    """A configuration drawn at random: two to six layers of either kind with any sizes (with ``tensor_core`` multiples of
    eight), windows from 1 to 300 or none, any feed-forward or none."""
    width = rng.choice([64, 96, 192]) if tensor_core else rng.choice([24, 40, 57, 72, 100])
    pick = (lambda lo, hi: 8 * rng.randint(max(1, lo // 8), hi // 8)) if tensor_core else rng.randint
    layers = []
    for _ in range(rng.randint(2, 6)):
        if rng.random() < 0.5:
            layer = _latent(rng.randint(1, 24), pick(3, 48), 2 * rng.randint(1, 20) if not tensor_core else pick(8, 40), pick(3, 48),
                            pick(4, 64), pick(4, 160), rng.choice([None, 1, 2, 7, 16, 17, 31, 64, 100, 129, 200, 300]),
                            base=rng.choice([100.0, 10000.0, 1000000.0]))
            layer["mixer"]["scale"] *= rng.choice([1.0, 2.0])
        else:
            G = rng.choice([1, 2, 3])
            H, vd = G * rng.randint(1, 4), pick(3, 80)
            parts = rng.choice([p for p in range(1, 9) if (H * vd) % p == 0])
            layer = _mamba(H, vd, pick(3, 140), G, rng.randint(1, 6), parts)
        u = rng.random()
        if u < 0.2:
            layer = _ff(layer)
        elif u < 0.45:
            layer = _ff(layer, pick(6, 96))
        else:
            E = rng.randint(1, 12)
            layer = _ff(layer, pick(6, 40), E, rng.randint(1, min(E, 4)))
        layers.append(layer)
    return _model(rng.choice([97, 301, 523]), width, rng.choice([1e-6, 1e-5]), rng.choice([None, 0.25, 0.8, 1.4]), layers)


def tensor_shapes(cfg) -> Dict[str, tuple]:
    """Every tensor of a model of this design, by the naming rule of its checkpoints."""
    D, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, D), "final.norm": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out.update({p + "norm1": (D,), p + "shift": (D,)})
        H, vd = m["heads"], m["vdim"]
        if layer["type"] == "latent_attention":
            d, rd, qr, r = m["dim"], m["rot_dim"], m["q_rank"], m["kv_rank"]
            out.update({p + "mix.dq": (qr, D), p + "mix.dq.norm": (qr,), p + "mix.uq": (H * (d + rd), qr), p + "mix.dkv": (r + rd, D),
                        p + "mix.dkv.norm": (r,), p + "mix.uk": (H * d, r), p + "mix.uv": (H * vd, r), p + "mix.o": (D, H * vd)})
        else:
            inner, gn = H * vd, m["groups"] * m["state"]
            out.update({p + "mix.in": (2 * inner + 2 * gn + H, D), p + "mix.conv": (inner + 2 * gn, m["conv"]),
                        p + "mix.conv.b": (inner + 2 * gn,), p + "mix.dt_bias": (H,), p + "mix.A_log": (H,), p + "mix.D": (H,),
                        p + "mix.norm": (inner,), p + "mix.o": (D, inner)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        out[p + "norm2"] = (D,)
        if mlp["kind"] == "dense":
            out.update({p + "mlp.up": (mlp["ff"], D), p + "mlp.down": (D, mlp["ff"])})
        else:
            E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            out.update({p + "mlp.router": (E, D), p + "mlp.router.b": (E,)})
            for e in range(E):
                out.update({p + f"mlp.e{e}.gate": (ff, D), p + f"mlp.e{e}.up": (ff, D), p + f"mlp.e{e}.down": (D, ff)})
    return out


def random_weights(cfg, seed: int, store=torch.float32, fixed_choice: bool = False) -> Dict[str, torch.Tensor]:
    """Weights that keep activations of order one: matrices N(0, 1/in), norm weights around zero where the design adds 1 and
    around one elsewhere, decays that forget within a few to a few hundred tokens.  ``fixed_choice``: small router rows and
    biases 1.5 apart in a random order, so that no rounding flips which experts are chosen.  Rounded once to ``store``."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        tail = name.split(".")[-1]
        rn = torch.randn(shape, generator=g)
        if tail in ("norm1", "norm2") or name == "final.norm":
            t = 0.1 * rn
        elif tail in ("norm", "D"):
            t = 1.0 + 0.1 * rn
        elif tail == "shift":
            t = 0.3 + 0.3 * rn
        elif name.endswith("router.b"):
            t = 1.5 * torch.randperm(shape[0], generator=g).float() if fixed_choice else 0.5 * rn
        elif tail == "router":
            t = (0.2 if fixed_choice else 2.0) * rn / shape[1] ** 0.5
        elif tail == "dt_bias":
            t = -2.0 + rn
        elif tail == "A_log":
            t = -0.5 + rn
        elif tail in ("conv", "b"):
            t = 0.5 * rn
        elif name == "embed":
            t = rn
        else:
            t = rn / shape[1] ** 0.5
        out[name] = t.to(store).contiguous()
    return out


def write_model(cfg, weights, out_dir: str) -> str:
    from lightllm_b200.weights import save_file
    os.makedirs(out_dir, exist_ok=True)
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(weights, os.path.join(out_dir, "model.safetensors"))
    return out_dir
