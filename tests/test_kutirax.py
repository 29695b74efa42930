"""Kutirax without a device: the configuration, tensor names and cache needs as the engine derives them against a restatement
of the design's rules, and the plain functions against other formulations of the same mechanisms."""
import itertools
import math
import random

import pytest
import torch

from lightllm_b200.config import ConfigError, config_from_dict, model_spec_for
from lightllm_b200.models import Model
from tests.kutirax_configs import CONFIGS, config, random_config, random_weights, tensor_shapes
from tests.plain import kutirax_plain as P


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_and_shapes_follow_the_naming_rule(name):
    cfg = config(name)
    model = Model(model_spec_for(config_from_dict(cfg)))
    assert {s.name: tuple(s.shape) for s in model.weight_specs()} == tensor_shapes(cfg)
    assert model.graph_safe()


def test_random_configurations_build():
    for seed in range(40):
        cfg = random_config(random.Random(seed), seed % 2 == 0)
        model = Model(model_spec_for(config_from_dict(cfg)))
        assert {s.name: tuple(s.shape) for s in model.weight_specs()} == tensor_shapes(cfg)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_cache_needs_of_every_layer(name):
    """A latent layer keeps one key row a token (the latent and the rotated part, no values); a recurrent one its states and
    its convolution's last inputs; every layer its last normed input."""
    cfg = config(name)
    layout = Model(model_spec_for(config_from_dict(cfg))).cache_layout
    assert len(layout.refs) == len(cfg["layers"]) == len(layout.state_planes)
    for ref, layer in zip(layout.refs, cfg["layers"]):
        m, floats = layer["mixer"], cfg["width"]
        if layer["type"] == "latent_attention":
            kv = layout.groups[ref.group]
            assert (kv.kv_heads, kv.head_dim, kv.value_dim, kv.window) == (1, m["kv_rank"] + m["rot_dim"], 0, (m.get("mask") or {}).get("size"))
        else:
            assert ref.group is None
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            floats += m["heads"] * m["state"] * m["vdim"] + (m["conv"] - 1) * (inner + 2 * gn)
        assert math.prod(layout.state_planes[ref.state_plane].shape) == floats


def test_layers_are_parallel_with_two_norms_and_a_shift_before_the_mixer():
    spec = model_spec_for(config_from_dict(config("A")))
    for i, layer in enumerate(spec.layers):
        assert layer.arrangement == "parallel" and layer.branch_scale == 0.7
        assert layer.sub_blocks[0].input_filter.kind == "token_shift" and layer.sub_blocks[0].norm_before.params["weight_name"] == f"l{i}.norm1"
        assert all(sb.norm_before.params["one_plus"] for sb in layer.sub_blocks)
    assert [len(l.sub_blocks) for l in spec.layers] == [2, 2, 1, 2]                     # mlp: null
    assert spec.layers[1].sub_blocks[1].norm_before.params["weight_name"] == "l1.norm2" and spec.layers[1].sub_blocks[1].input_filter is None
    assert spec.head.params["weight_name"] == "embed"
    none = model_spec_for(config_from_dict(config("C")))
    assert none.layers[0].branch_scale == 1.0 and none.layers[2].sub_blocks[0].part.params["window"] is None


def test_configuration_errors_name_the_key():
    def broken(edit):
        cfg = config("A")
        edit(cfg)
        return cfg
    cases = [
        (lambda c: c.pop("vocab"), "vocab"),
        (lambda c: c["norm"].pop("eps"), "eps"),
        (lambda c: c["layers"][0].update(type="serial"), "type"),
        (lambda c: c["layers"][0]["mixer"].update(groups=2), "groups"),
        (lambda c: c["layers"][0]["mixer"].update(norm_groups=4), "norm_groups"),
        (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
        (lambda c: c["layers"][0]["mixer"].pop("state"), "state"),
        (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind"),
        (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
        (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
        (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4), "dims"),
        (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
        (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top"),
        (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
        (lambda c: c.update(layers=[]), "layers"),
    ]
    for edit, word in cases:
        with pytest.raises(ConfigError) as e:
            config_from_dict(broken(edit))
        assert word in str(e.value), (word, str(e.value))


# ---- the plain functions against other formulations -----------------------------------------------------------------
def test_plain_shift_is_a_convolution_of_two_taps():
    torch.manual_seed(0)
    h, mix = torch.randn(9, 5, dtype=P.F), torch.randn(5, dtype=P.F)
    w = torch.stack([mix, 1 - mix], 1)
    assert torch.allclose(P.token_shift(h, mix), P.causal_conv(h, w, torch.zeros(5, dtype=P.F)), atol=1e-12)


def test_plain_convolution_equals_conv1d():
    torch.manual_seed(1)
    u, w, b = torch.randn(11, 6, dtype=P.F), torch.randn(6, 4, dtype=P.F), torch.randn(6, dtype=P.F)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T[None], (3, 0)), w[:, None], b, groups=6)[0].T
    assert torch.allclose(P.causal_conv(u, w, b), want, atol=1e-12)


def test_plain_rotation_is_a_complex_product_and_keeps_relative_positions():
    torch.manual_seed(2)
    x = torch.randn(7, 3, 8, dtype=P.F)
    y = P.rotate(x, 100.0, 8)
    f = 100.0 ** (-torch.arange(4, dtype=P.F) / 4)
    z = torch.complex(x[..., :4], x[..., 4:]) * torch.polar(torch.ones(7, 4, dtype=P.F), torch.arange(7, dtype=P.F)[:, None] * f)[:, None]
    assert torch.allclose(y, torch.cat([z.real, z.imag], -1), atol=1e-12)
    same = x[:1].expand(7, 3, 8)
    r = P.rotate(same.clone(), 100.0, 8)
    assert torch.allclose((r[5] * r[3]).sum(-1), (r[4] * r[2]).sum(-1), atol=1e-12)


def test_plain_latent_attention_equals_attention_over_the_cached_rows():
    """The up-projections moved onto the query and the output: multi-query attention over rows [latent | rotated part] whose
    first numbers are the values."""
    torch.manual_seed(3)
    cfg = config("A")
    m, eps, p = cfg["layers"][1]["mixer"], 1e-5, "l1.mix"
    t = {k: v.double() for k, v in random_weights(cfg, 2).items()}
    T, H, d, rd, vd, r = 30, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    h = torch.randn(T, cfg["width"], dtype=P.F)
    got = P.latent_attention(h, m, t, p, eps)
    cq = P.unit_rms(h @ t[f"{p}.dq"].T, eps) * t[f"{p}.dq.norm"]
    q = (cq @ t[f"{p}.uq"].T).view(T, H, d + rd)
    down = h @ t[f"{p}.dkv"].T
    rows = torch.cat([P.unit_rms(down[:, :r], eps) * t[f"{p}.dkv.norm"], P.rotate(down[:, r:], m["rot"]["base"], rd)], -1)
    qq = torch.cat([torch.einsum("thd,hdr->thr", q[..., :d], t[f"{p}.uk"].view(H, d, r)), P.rotate(q[..., d:], m["rot"]["base"], rd)], -1)
    s = torch.einsum("ihw,jw->hij", qq, rows) * m["scale"]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    s = s.masked_fill(~((j <= i) & (i - j < m["mask"]["size"])), -math.inf)
    mixed = torch.einsum("hij,jr->ihr", torch.softmax(s, -1), rows[:, :r])
    out = torch.einsum("ihr,hvr->ihv", mixed, t[f"{p}.uv"].view(H, vd, r)).reshape(T, H * vd) @ t[f"{p}.o"].T
    assert torch.allclose(got, out, atol=1e-11)


def test_plain_recurrence_equals_the_masked_product():
    """``y_t = sum_{s <= t} (C_t . B_s) exp(sum of the log decays after s) dt_s x_s + D x_t``."""
    torch.manual_seed(4)
    T, H, G, N, vd = 17, 4, 2, 5, 3
    x, B, C = torch.randn(T, H, vd, dtype=P.F), torch.randn(T, G, N, dtype=P.F), torch.randn(T, G, N, dtype=P.F)
    dt, A, D = torch.rand(T, H, dtype=P.F), torch.randn(H, dtype=P.F), torch.randn(H, dtype=P.F)
    got = P.state_space(x, B, C, dt, A, D)
    L = torch.cumsum(-torch.exp(A) * dt, 0)
    for h in range(H):
        g = h // (H // G)
        M = (C[:, g] @ B[:, g].T) * torch.exp(L[:, None, h] - L[None, :, h]) * dt[None, :, h]
        want = torch.tril(M) @ x[:, h] + D[h] * x[:, h]
        assert torch.allclose(got[:, h], want, atol=1e-12)


def test_plain_gated_norm_by_parts():
    torch.manual_seed(5)
    y, z, w = torch.randn(4, 12, dtype=P.F), torch.randn(4, 12, dtype=P.F), torch.randn(12, dtype=P.F)
    got = P.gated_group_norm(y, z, w, 3, 1e-5)
    for part in range(3):
        sl = slice(4 * part, 4 * part + 4)
        g = y[:, sl] * torch.nn.functional.silu(z[:, sl])
        assert torch.allclose(got[:, sl], g / (g.pow(2).mean(-1, keepdim=True) + 1e-5).sqrt() * w[sl], atol=1e-12)


def test_plain_routing_by_brute_force():
    torch.manual_seed(6)
    D, E, top = 16, 6, 3
    W, b, h = torch.randn(E, D, dtype=P.F), torch.randn(E, dtype=P.F), torch.randn(20, D, dtype=P.F)
    ids, wts = P.route(h, W, b, top)
    z = h @ W.T + b
    for t in range(20):
        best = max(itertools.combinations(range(E), top), key=lambda es: sum(float(z[t, e]) for e in es))
        assert sorted(ids[t].tolist()) == sorted(best)
        total = sum(math.exp(float(z[t, e])) for e in best)
        for e, w in zip(ids[t].tolist(), wts[t]):
            assert abs(float(w) - math.exp(float(z[t, e])) / total) < 1e-12


def test_plain_model_runs_every_configuration():
    for name in CONFIGS:
        cfg = config(name)
        w = random_weights(cfg, 1)
        streams = []
        logits = P.forward(cfg, w, list(range(3, 30)), streams)
        assert logits.shape == (27, cfg["vocab"]) and len(streams) == len(cfg["layers"]) and bool(torch.isfinite(logits).all())
        # causal: a position's logits do not change with what follows
        assert torch.allclose(P.forward(cfg, w, list(range(3, 20))), logits[:17], atol=1e-10)
