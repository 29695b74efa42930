"""``Laralix``: a pre-norm decoder (``h += mixer(norm(h)); h += ff(norm(h))``, RMS norms whose weight is stored around zero and
applied as ``1 + w``) whose layers each pick one of three mixers:

* ``parallel``: windowed attention with a bias by distance (head-normed q and k, soft-capped scores, one added to the softmax's
  sum; :class:`~lightllm_b200.parts.distance_attention.DistanceAttentionMixer`) beside the gated delta rule with one decay a head
  (:class:`~lightllm_b200.parts.delta.HeadDeltaMixer`), the mean of the two outputs, each RMS-normed;
* ``parallel_2``: attention over a window and the first tokens whose values are its keys as projected, q and k normed over their
  whole projection (:class:`~lightllm_b200.parts.sink_attention.KeyValuedAttentionMixer`), beside gated linear attention
  (:class:`~lightllm_b200.parts.gated_linear.GatedLinearMixer`), a weighted sum of the two outputs;
* ``latent_attention``: attention over a cached latent with a rotated key part shared by all heads
  (:class:`~lightllm_b200.parts.rotary_latent_attention.RotaryLatentAttentionMixer`).

Feed-forwards are gated by SiLU.  A stretch of layers may run several times in a row with the same weights: a learned vector is
added to the stream before every pass, and before every pass but the first the embedding output as well; every pass has cache
and state of its own.  The embedding and the logits are multiplied by constants.

config.json: ``architecture`` (the name), ``vocab``, ``width``, ``embedding.scale``, ``logit_scale``, ``norm.eps``, ``loop``
``{"start", "stop", "times"}`` and ``layers``, a list of ``{"type", "mixer": {...}, "mlp": {"kind": "dense", "ff"} | null}`` with the
mixers ``{"left": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask": {"size"}}, "right": {"heads", "kv_heads", "dim",
"vdim", "conv"}}``, ``{"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "keep_first"}}, "right": {"heads",
"dim", "vdim", "tau"}, "left_scale", "right_scale"}`` and ``{"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot":
{"base", "dims"}}``.  The rank of the decays' low-rank pair is the row count of ``l<i>.mix.right.a1`` in the checkpoint (a
configuration that is not read beside a checkpoint gives it as ``decay_rank`` in the right mixer's object).

Tensors: ``embed``, ``head``, ``final.norm``, ``loop.step`` and per layer i ``l<i>.norm1|norm2``, ``l<i>.mix.left.q|k|v|o|q.norm|k.norm|out``,
``l<i>.mix.right.q|k|v|b|a|g|o|q.conv|k.conv|v.conv|A_log|dt_bias|norm|out`` (or ``a1|a2|a2.b`` in the place of ``b|a`` and what
belongs to them), ``l<i>.mix.dq|uq|dkv|uk|uv|o`` (+ ``.norm`` on dq and dkv), ``l<i>.mlp.gate|up|down``; linear weights are
``[out, in]`` without a ``.weight`` ending.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..config import (ConfigError, ConfigReader, LayerSpec, ModelConfig, ModelSpec, PartSpec, RunEntry, SubBlock,
                      architecture_name, register_architecture)

# Rotations are computed from the position itself; the engine only wants a bound for its buffers.
MAX_POSITIONS = 1 << 20
MIXER_TYPES = ("parallel", "parallel_2", "latent_attention")
# One is added to the softmax's sum: a sink whose score is 0.
SINK_SCORE = 0.0


def _object(raw: Any, key: str, where: str, required: bool = True) -> Optional[Dict[str, Any]]:
    v = raw.get(key)
    if v is None and not required:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: {'required ' if required else ''}key '{key}' must be an object")
    return v


@dataclass(frozen=True)
class LaralixLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


def _grouped(r: ConfigReader, where: str) -> Dict[str, Any]:
    out = {k: r.integer(k) for k in ("heads", "kv_heads", "dim")}
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"{where}: 'heads' {out['heads']} is not a multiple of 'kv_heads' {out['kv_heads']}")
    return out


def _mask(raw: Dict[str, Any], where: str, out: Dict[str, Any], keeps: bool) -> None:
    out["window"], out["keep_first"] = None, 0
    mask = _object(raw, "mask", where, required=False)
    if mask is not None:
        r = ConfigReader(mask, f"{where}.mask")
        out["window"] = r.integer("size")
        if keeps:
            out["keep_first"] = r.integer("keep_first", 0, minimum=0)


def _parallel(raw: Dict[str, Any], where: str) -> Dict[str, Any]:
    lraw, rraw = _object(raw, "left", where), _object(raw, "right", where)
    lr, rr = ConfigReader(lraw, f"{where}.left"), ConfigReader(rraw, f"{where}.right")
    left = _grouped(lr, f"{where}.left")
    left.update(vdim=lr.integer("vdim"), scale=lr.real("scale"),
                softcap=lr.real("softcap") if lraw.get("softcap") is not None else None)
    _mask(lraw, f"{where}.left", left, keeps=False)
    right = _grouped(rr, f"{where}.right")
    right.update(vdim=rr.integer("vdim"), conv=rr.integer("conv", None))          # no 'conv': no convolution
    return {"left": left, "right": right}


def _parallel_2(raw: Dict[str, Any], where: str, index: int, shapes: Optional[Dict[str, tuple]]) -> Dict[str, Any]:
    lraw, rraw = _object(raw, "left", where), _object(raw, "right", where)
    lr, rr, r = ConfigReader(lraw, f"{where}.left"), ConfigReader(rraw, f"{where}.right"), ConfigReader(raw, where)
    left = _grouped(lr, f"{where}.left")
    left["scale"] = lr.real("scale")
    if lr.integer("vdim", left["dim"]) != left["dim"]:
        raise ConfigError(f"{where}.left: the values are the keys, but 'vdim' {lraw['vdim']} is not 'dim' {left['dim']}")
    _mask(lraw, f"{where}.left", left, keeps=True)
    right: Dict[str, Any] = {k: rr.integer(k) for k in ("heads", "dim", "vdim")}
    right["tau"] = rr.real("tau")
    name = f"l{index}.mix.right.a1"
    if rraw.get("decay_rank") is not None:
        right["decay_rank"] = rr.integer("decay_rank")
    elif shapes is not None and name in shapes and len(shapes[name]) == 2:
        right["decay_rank"] = int(shapes[name][0])
    else:
        raise ConfigError(f"{where}.right: the rank 'decay_rank' is neither in the configuration nor given by the shape of a "
                          f"tensor '{name}' in a checkpoint beside it")
    return {"left": left, "right": right, "left_scale": r.real("left_scale", positive=False),
            "right_scale": r.real("right_scale", positive=False)}


def _latent(raw: Dict[str, Any], where: str) -> Dict[str, Any]:
    r = ConfigReader(raw, where)
    out: Dict[str, Any] = {k: r.integer(k) for k in ("heads", "dim", "vdim", "q_rank", "kv_rank")}
    out["rot_dim"] = r.integer("rot_dim", minimum=2)
    out["scale"] = r.real("scale")
    rr = ConfigReader(_object(raw, "rot", where), f"{where}.rot")
    dims = rr.integer("dims", out["rot_dim"])
    if dims % 2 or dims != out["rot_dim"]:
        raise ConfigError(f"{where}.rot: 'dims' {dims} must be even and equal to 'rot_dim' {out['rot_dim']}")
    out["base"] = rr.real("base")
    return out


@dataclass(frozen=True)
class LaralixConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-5
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    layers: Tuple[LaralixLayer, ...] = field(default_factory=tuple)
    loop: Optional[Tuple[int, int, int]] = None          # (start, stop, times)

    @staticmethod
    def from_dict(raw: Dict[str, Any], where: str = "config.json",
                  tensor_shapes: Optional[Dict[str, tuple]] = None) -> "LaralixConfig":
        r = ConfigReader(raw, where)
        arch = architecture_name(raw, where)
        norm = ConfigReader(_object(raw, "norm", where), f"{where}: norm")
        emb = _object(raw, "embedding", where, required=False)
        scale = ConfigReader(emb, f"{where}: embedding").real("scale", 1.0, positive=False) if emb is not None else 1.0
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError(f"{where}: required key 'layers' must be a non-empty list")
        layers: List[LaralixLayer] = []
        raw_layers: List[Dict[str, Any]] = []
        for i, lr in enumerate(layers_raw):
            w = f"{where}: layers[{i}]"
            if not isinstance(lr, dict):
                raise ConfigError(f"{w} must be an object")
            kind = ConfigReader(lr, w).string("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{w}: unknown 'type' {kind!r}; known: {list(MIXER_TYPES)}")
            m, mw = _object(lr, "mixer", w), f"{w}.mixer"
            if kind == "parallel":
                mixer = _parallel(m, mw)
            elif kind == "parallel_2":
                mixer = _parallel_2(m, mw, i, tensor_shapes)
                # the rank read from a tensor's shape is written back, so that the configuration stands on its own
                lr = dict(lr, mixer=dict(m, right=dict(m["right"], decay_rank=mixer["right"]["decay_rank"])))
            else:
                mixer = _latent(m, mw)
            mlp = _object(lr, "mlp", w, required=False)
            if mlp is not None:
                mr = ConfigReader(mlp, f"{w}.mlp")
                if mr.string("kind") != "dense":
                    raise ConfigError(f"{w}.mlp: 'kind' must be 'dense', got {mlp['kind']!r}")
                mlp = {"ff": mr.integer("ff")}
            layers.append(LaralixLayer(kind, mixer, mlp))
            raw_layers.append(lr)
        loop = None
        lp = _object(raw, "loop", where, required=False)
        if lp is not None:
            lpr = ConfigReader(lp, f"{where}: loop")
            start, stop, times = lpr.integer("start", minimum=0), lpr.integer("stop", minimum=0), lpr.integer("times")
            if not start <= stop <= len(layers):
                raise ConfigError(f"{where}: loop: layers {start} .. {stop} - 1 are not a stretch of the {len(layers)} layers")
            loop = (start, stop, times) if stop > start else None          # an empty stretch: nothing is run again
        return LaralixConfig(architecture=arch, raw=dict(raw, layers=raw_layers), vocab=r.integer("vocab"), width=r.integer("width"),
                             norm_eps=norm.real("eps", positive=False), embedding_scale=scale,
                             logit_scale=r.real("logit_scale", 1.0, positive=False), layers=tuple(layers), loop=loop)


def _mixer_spec(layer: LaralixLayer, p: str, D: int, eps: float) -> PartSpec:
    """``p``: where the mixer's tensors live (``l<i>.mix``)."""
    m, plain = layer.mixer, {"weight_suffix": ""}
    if layer.type == "latent_attention":
        rot = PartSpec("rotary", {"head_dim": m["rot_dim"], "theta": m["base"], "rotary_dim": m["rot_dim"], "style": "interleaved"})
        return PartSpec("rotary_latent_attention", {
            "hidden_size": D, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "v_head_dim": m["vdim"],
            "q_rank": m["q_rank"], "rank": m["kv_rank"], "position": rot, "norm_eps": eps, "scale": m["scale"],
            "names": {n: n for n in ("dq", "uq", "dkv", "uk", "uv", "o")}, **plain}, p)
    a, b = m["left"], m["right"]
    attention = {"hidden_size": D, "num_heads": a["heads"], "num_kv_heads": a["kv_heads"], "head_dim": a["dim"], "window": a["window"],
                 "scale": a["scale"], **plain}
    recurrence = {"hidden_size": D, "num_heads": b["heads"], "head_dim": b["dim"], "v_head_dim": b["vdim"], "norm_eps": eps, **plain}
    if layer.type == "parallel":
        left = PartSpec("distance_attention", {
            **attention, "v_head_dim": a["vdim"], "softcap": a["softcap"], "sink": SINK_SCORE, "qk_norm": True, "norm_eps": eps,
            "names": {n: n for n in "qkvo"}}, f"{p}.left")
        right = PartSpec("head_delta", {
            **recurrence, "num_qk_heads": b["kv_heads"], "conv_taps": b["conv"] or 0, "conv_ending": "conv",
            "names": {n: n for n in ("q", "k", "v", "b", "a", "g", "o", "A_log", "dt_bias", "norm")}}, f"{p}.right")
        return PartSpec("joined_mixers", {"hidden_size": D, "mixers": [left, right], "eps": eps,
                                          "out_norms": [f"{p}.left.out", f"{p}.right.out"], "weights": [0.5, 0.5]}, p)
    left = PartSpec("key_valued_attention", {
        **attention, "keep_first": a["keep_first"], "sinks": False, "gate": False, "qk_bias": False, "qk_norm": "projection",
        "qk_norm_eps": eps, "names": {n: n for n in "qko"}}, f"{p}.left")
    right = PartSpec("gated_linear_attention", {
        **recurrence, "decay_rank": b["decay_rank"], "tau": b["tau"], "bias_ending": "b",
        "names": {n: n for n in ("q", "k", "v", "g", "o", "a1", "a2", "norm")}}, f"{p}.right")
    return PartSpec("joined_mixers", {"hidden_size": D, "mixers": [left, right], "eps": eps, "out_norms": None,
                                      "weights": [m["left_scale"], m["right_scale"]]}, p)


def laralix_spec(cfg: LaralixConfig) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"hidden_size": D, "eps": eps, "weight_name": "", "one_plus": True}, name)

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}"
        subs = [SubBlock("mixer", _mixer_spec(layer, f"{p}.mix", D, eps), norm_before=norm(f"{p}.norm1"))]
        if layer.mlp is not None:
            ffn = PartSpec("gated_mlp", {"hidden_size": D, "intermediate_size": layer.mlp["ff"], "activation": "silu",
                                         "names": {n: n for n in ("gate", "up", "down")}, "weight_suffix": ""}, f"{p}.mlp")
            subs.append(SubBlock("ffn", ffn, norm_before=norm(f"{p}.norm2")))
        layers.append(LayerSpec(sub_blocks=subs, arrangement="sequential"))

    n = len(layers)
    start, stop, times = cfg.loop if cfg.loop is not None else (n, n, 0)
    run = [RunEntry(i) for i in range(start)]
    for t in range(times):
        enter = PartSpec("step_vector", {"hidden_size": D, "step_name": "loop.step", "steps": times, "index": t,
                                         "add_embedding": t > 0}, "")
        run += [RunEntry(i, enter=enter if i == start else None) for i in range(start, stop)]
    run += [RunEntry(i) for i in range(stop, n)]
    # a layer without a feed-forward does not read the norm, nor a model without a loop the step vectors, that a checkpoint may carry
    ignored = tuple(f"l{i}.norm2" for i, layer in enumerate(cfg.layers) if layer.mlp is None)
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=D, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": D, "weight_name": "embed",
                                               "scale": cfg.embedding_scale,
                                               "keep_output": "float32" if times > 1 else False}, ""),
        layers=layers, run=run, final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": D, "weight_name": "head", "scale": cfg.logit_scale}, ""),
        ignored_suffixes=ignored + (("loop.step",) if cfg.loop is None else ()))


register_architecture("Laralix", LaralixConfig.from_dict, laralix_spec, reads_shapes=True)
