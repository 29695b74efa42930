"""``Kutirax``: a decoder of parallel layers, ``x += m * (mixer(shift(norm1(x))) + ff(norm2(x)))``, both branches of the same x
and each with an RMS norm of its own whose weight is stored around zero.  What the mixer reads is first moved towards the
token before, ``h + (h_before - h) * mix`` (a request's last h is part of its state in every layer).

Mixers: ``latent_attention`` (queries and keys/values through low-rank latents, rotary positions on a part of the queries and
on one key part shared by all heads, a sliding window) and ``mamba2`` (the state-space recurrence with a short convolution, a
SiLU gate and a group norm).  Feed-forwards: dense with the square of relu, or routed experts whose weights are the softmax
over the chosen logits.  The logits come from the embedding table.

config.json: ``architecture`` (the name), ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` and ``layers``, a list of ``{"type",
"mixer": {...}, "mlp": {...} | null}`` with the mixers ``{"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot":
{"base", "dims"}, "mask": {"size"}}`` and ``{"heads", "vdim", "state", "groups", "conv", "norm_groups"}`` and the feed-forwards
``{"kind": "dense", "ff"}`` and ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}``.  No ``residual_mult`` is a
multiplier of 1, no ``mask`` every earlier key.  Tensors: ``embed``, ``final.norm`` and per layer i ``l<i>.norm1|norm2|shift``,
``l<i>.mix.dq|uq|dkv|uk|uv|o`` (+ ``.norm`` on dq and dkv) or ``l<i>.mix.in|conv|conv.b|dt_bias|A_log|D|norm|o``, ``l<i>.mlp.up|down`` or
``l<i>.mlp.router|router.b`` and ``l<i>.mlp.e<j>.gate|up|down``; linear weights are ``[out, in]`` without a ``.weight`` ending.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..config import (ConfigError, ConfigReader, LayerSpec, ModelConfig, ModelSpec, PartSpec, RunEntry, SubBlock,
                      architecture_name, register_architecture)

# The design has no table of positions; the engine only wants a bound for its buffers.
MAX_POSITIONS = 1 << 20
MIXER_TYPES = ("latent_attention", "mamba2")
FF_KINDS = ("dense", "moe")


def _object(raw: Any, key: str, where: str, required: bool = True) -> Optional[Dict[str, Any]]:
    v = raw.get(key)
    if v is None and not required:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: {'required ' if required else ''}key '{key}' must be an object")
    return v


@dataclass(frozen=True)
class KutiraxLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


@dataclass(frozen=True)
class KutiraxConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    layers: Tuple[KutiraxLayer, ...] = field(default_factory=tuple)

    @staticmethod
    def _latent(raw: Any, where: str) -> Dict[str, Any]:
        r = ConfigReader(raw, where)
        out: Dict[str, Any] = {k: r.integer(k) for k in ("heads", "dim", "vdim", "q_rank", "kv_rank")}
        out["rot_dim"] = r.integer("rot_dim", minimum=2)
        out["scale"] = r.real("scale", positive=False)
        rr = ConfigReader(_object(raw, "rot", where), f"{where}.rot")
        dims = rr.integer("dims", out["rot_dim"])
        if dims % 2 or dims != out["rot_dim"]:
            raise ConfigError(f"{where}.rot: 'dims' {dims} must be even and equal to 'rot_dim' {out['rot_dim']}")
        out["base"] = rr.real("base")
        mask = _object(raw, "mask", where, required=False)
        out["window"] = ConfigReader(mask, f"{where}.mask").integer("size") if mask is not None else None
        return out

    @staticmethod
    def _mamba2(raw: Any, where: str) -> Dict[str, Any]:
        r = ConfigReader(raw, where)
        out = {k: r.integer(k) for k in ("heads", "vdim", "state", "groups", "conv")}
        out["norm_groups"] = r.integer("norm_groups", 1)
        if out["heads"] % out["groups"]:
            raise ConfigError(f"{where}: 'heads' {out['heads']} is not a multiple of 'groups' {out['groups']}")
        if (out["heads"] * out["vdim"]) % out["norm_groups"]:
            raise ConfigError(f"{where}: {out['heads']} heads of {out['vdim']} do not fall into 'norm_groups' {out['norm_groups']} equal parts")
        return out

    @staticmethod
    def _mlp(raw: Any, where: str) -> Dict[str, Any]:
        r = ConfigReader(raw, where)
        kind = r.string("kind")
        if kind == "dense":
            return {"kind": kind, "ff": r.integer("ff")}
        if kind != "moe":
            raise ConfigError(f"{where}: unknown 'kind' {kind!r}; known: {list(FF_KINDS)}")
        er = ConfigReader(_object(raw, "expert", where), f"{where}.expert")
        rr = ConfigReader(_object(raw, "router", where), f"{where}.router")
        out = {"kind": kind, "ff": er.integer("ff"), "experts": rr.integer("experts"), "top": rr.integer("top")}
        if out["top"] > out["experts"]:
            raise ConfigError(f"{where}.router: 'top' {out['top']} of {out['experts']} experts")
        return out

    @staticmethod
    def from_dict(raw: Dict[str, Any], where: str = "config.json") -> "KutiraxConfig":
        r = ConfigReader(raw, where)
        arch = architecture_name(raw, where)
        norm = ConfigReader(_object(raw, "norm", where), f"{where}: norm")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError(f"{where}: required key 'layers' must be a non-empty list")
        layers: List[KutiraxLayer] = []
        for i, lr in enumerate(layers_raw):
            w = f"{where}: layers[{i}]"
            if not isinstance(lr, dict):
                raise ConfigError(f"{w} must be an object")
            kind = ConfigReader(lr, w).string("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{w}: unknown 'type' {kind!r}; known: {list(MIXER_TYPES)}")
            read = KutiraxConfig._latent if kind == "latent_attention" else KutiraxConfig._mamba2
            mlp = _object(lr, "mlp", w, required=False)
            layers.append(KutiraxLayer(kind, read(_object(lr, "mixer", w), f"{w}.mixer"),
                                       None if mlp is None else KutiraxConfig._mlp(mlp, f"{w}.mlp")))
        return KutiraxConfig(architecture=arch, raw=dict(raw), vocab=r.integer("vocab"), width=r.integer("width"),
                             norm_eps=norm.real("eps", positive=False), residual_mult=r.real("residual_mult", 1.0, positive=False),
                             layers=tuple(layers))


def kutirax_spec(cfg: KutiraxConfig) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps

    def rms(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"hidden_size": D, "eps": eps, "weight_name": name, "one_plus": True}, "")

    layers: List[LayerSpec] = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer.mixer
        if layer.type == "latent_attention":
            rot = PartSpec("rotary", {"head_dim": m["rot_dim"], "theta": m["base"], "rotary_dim": m["rot_dim"], "style": "neox"})
            mixer = PartSpec("rotary_latent_attention", {
                "hidden_size": D, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "v_head_dim": m["vdim"],
                "q_rank": m["q_rank"], "rank": m["kv_rank"], "position": rot, "norm_eps": eps, "scale": m["scale"],
                "window": m["window"], "names": {n: n for n in ("dq", "uq", "dkv", "uk", "uv", "o")}, "weight_suffix": ""},
                f"{p}.mix")
        else:
            mixer = PartSpec("state_space", {
                "hidden_size": D, "num_heads": m["heads"], "v_head_dim": m["vdim"], "state_dim": m["state"], "groups": m["groups"],
                "conv_taps": m["conv"], "norm_groups": m["norm_groups"], "norm_eps": eps,
                "names": {"in": "in", "conv": "conv", "o": "o"}, "weight_suffix": "", "bias_ending": "b"}, f"{p}.mix")
        shift = PartSpec("token_shift", {"channels": D, "weight_name": ""}, f"{p}.shift")
        subs = [SubBlock("mixer", mixer, norm_before=rms(f"{p}.norm1"), input_filter=shift)]
        if layer.mlp is not None:
            f = layer.mlp
            if f["kind"] == "dense":
                ffn = PartSpec("plain_mlp", {"hidden_size": D, "intermediate_size": f["ff"], "activation": "squared_relu",
                                             "names": {"up": "up", "down": "down"}, "weight_suffix": ""}, f"{p}.mlp")
            else:
                ffn = PartSpec("routed_experts", {
                    "hidden_size": D, "intermediate_size": f["ff"], "num_experts": f["experts"], "top": f["top"],
                    "score": "softmax_chosen", "router_bias": True, "bias_ending": "b",
                    "names": {"gate": "gate", "up": "up", "down": "down", "router": "router"}, "weight_suffix": "",
                    "expert_prefix": "e"}, f"{p}.mlp")
            subs.append(SubBlock("ffn", ffn, norm_before=rms(f"{p}.norm2")))
        layers.append(LayerSpec(sub_blocks=subs, arrangement="parallel", branch_scale=cfg.residual_mult))

    return ModelSpec(
        architecture=cfg.architecture, hidden_size=D, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": D, "weight_name": "embed"}, ""),
        layers=layers, run=[RunEntry(i) for i in range(len(layers))], final_norm=rms("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": D, "weight_name": "embed"}, ""),
        # a layer without a feed-forward does not read the norm that a checkpoint may carry for it
        ignored_suffixes=tuple(f"l{i}.norm2" for i, layer in enumerate(cfg.layers) if layer.mlp is None))


register_architecture("Kutirax", KutiraxConfig.from_dict, kutirax_spec)
