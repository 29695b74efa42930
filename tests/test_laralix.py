"""Laralix without a device: the configuration, tensor names, run list and cache needs as the engine derives them against a
restatement of the design's rules, pages of first tokens that stay while a window passes, and the plain functions against other
formulations of the same mechanisms."""
import math
import random

import pytest
import torch

from lightllm_b200.cache import CacheLayout, CacheManager, CacheSpec, KVSpec
from lightllm_b200.config import ConfigError, config_from_dict, load_config, model_spec_for
from lightllm_b200.models import Model
from tests.laralix_configs import CONFIGS, config, random_config, random_weights, tensor_shapes, write_model
from tests.plain import laralix_plain as P


def build(cfg):
    return Model(model_spec_for(config_from_dict(cfg)))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_and_shapes_follow_the_naming_rule(name):
    cfg = config(name)
    model = build(cfg)
    assert {s.name: tuple(s.shape) for s in model.weight_specs()} == tensor_shapes(cfg)
    assert model.graph_safe()


def test_random_configurations_build():
    for seed in range(40):
        cfg = random_config(random.Random(seed), seed % 2 == 0)
        assert {s.name: tuple(s.shape) for s in build(cfg).weight_specs()} == tensor_shapes(cfg)


def test_the_decays_rank_comes_from_the_checkpoint(tmp_path):
    cfg = config("A")
    d = write_model(cfg, random_weights(cfg, 1), str(tmp_path / "m"))
    read = load_config(d)
    assert read.layers[1].mixer["right"]["decay_rank"] == 3
    assert read.to_json_dict()["layers"][1]["mixer"]["right"]["decay_rank"] == 3          # written back
    again = config_from_dict(read.to_json_dict())
    assert again.layers == read.layers


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_run_list_and_what_enters_a_pass(name):
    cfg = config(name)
    spec = build(cfg).spec
    want = P.run_list(cfg)
    assert [e.layer for e in spec.run] == [i for i, _ in want]
    for e, (_, opens) in zip(spec.run, want):
        assert e.cache_of is None and (e.enter is not None) == (opens is not None)
        if opens is not None:
            assert (e.enter.params["index"], e.enter.params["add_embedding"]) == (opens, opens > 0)
    times = (cfg.get("loop") or {"times": 0})["times"]
    assert spec.embedding.params["keep_output"] == ("float32" if times > 1 else False)
    assert spec.head.params["scale"] == cfg["logit_scale"] and spec.embedding.params["scale"] == cfg["embedding"]["scale"]


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_cache_needs_of_every_run(name):
    """Every pass of the loop has pages and state of its own."""
    cfg = config(name)
    layout = build(cfg).cache_layout
    runs = P.run_list(cfg)
    assert len(layout.refs) == len(runs)
    seen = set()
    for ref, (i, _) in zip(layout.refs, runs):
        layer = cfg["layers"][i]
        m, kv = layer["mixer"], layout.groups[ref.group]
        assert (ref.group, ref.plane) not in seen
        seen.add((ref.group, ref.plane))
        if layer["type"] == "latent_attention":
            assert (kv.kv_heads, kv.head_dim, kv.value_dim, kv.window, ref.state_plane) == (1, m["kv_rank"] + m["rot_dim"], 0, None, None)
            continue
        a, b = m["left"], m["right"]
        mask = a.get("mask") or {}
        assert (kv.kv_heads, kv.head_dim, kv.value_dim) == (a["kv_heads"], a["dim"], a["vdim"])
        assert (kv.window, kv.keep_first) == (mask.get("size"), mask.get("keep_first", 0))
        floats = b["heads"] * b["dim"] * b["vdim"]
        if layer["type"] == "parallel":
            floats += (b["conv"] - 1) * (2 * b["kv_heads"] * b["dim"] + b["heads"] * b["vdim"])
        assert math.prod(layout.state_planes[ref.state_plane].shape) == floats


def test_configuration_errors_name_the_key():
    cases = [
        (lambda c: c.pop("vocab"), "vocab"),
        (lambda c: c["norm"].pop("eps"), "eps"),
        (lambda c: c["layers"][0].update(type="serial"), "type"),
        (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
        (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
        (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), "softcap"),
        (lambda c: c["layers"][0]["mixer"]["right"].update(conv=0), "conv"),
        (lambda c: c["layers"][0]["mixer"]["right"].update(kv_heads=3), "kv_heads"),
        (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
        (lambda c: c["layers"][1]["mixer"]["left"].update(vdim=5), "vdim"),
        (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first"),
        (lambda c: c["layers"][1]["mixer"]["right"].update(tau=0.0), "tau"),
        (lambda c: c["layers"][1]["mixer"]["right"].pop("decay_rank"), "decay_rank"),
        (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
        (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=4), "dims"),
        (lambda c: c["layers"][3]["mlp"].update(kind="moe"), "kind"),
        (lambda c: c["loop"].update(stop=9), "loop"),
        (lambda c: c["loop"].pop("times"), "times"),
        (lambda c: c.update(layers=[]), "layers"),
    ]
    for edit, word in cases:
        cfg = config("A")
        edit(cfg)
        with pytest.raises(ConfigError) as e:
            config_from_dict(cfg)
        assert word in str(e.value), (word, str(e.value))


# ---- the cache: first tokens stay ----------------------------------------------------------------------------------
@pytest.mark.parametrize("keep,window,page", [(3, 9, 4), (4, 9, 4), (5, 1, 4), (1, 16, 8), (0, 9, 4), (30, 7, 4)])
def test_pages_of_the_first_tokens_stay_while_the_window_passes(keep, window, page):
    layout = CacheLayout.build([CacheSpec(kv=KVSpec(1, 2, window, None, None, keep))], [None])
    m = CacheManager(layout, page, 40, 2, 160)
    rng = random.Random(keep * 100 + window)
    m.open("a")
    n = 0
    while n < 120:
        c = min(rng.choice([1, 1, 2, 5, 17]), 120 - n)
        m.reserve("a", c)
        m.advance("a", c)
        n += c
        table = m.block_table("a", 0)
        for lp in range(len(table)):          # a page is held exactly when the next query (or a later one) can see a position of it
            live = any(P.visible(n, p, window, keep) for p in range(lp * page, (lp + 1) * page) if p <= n) or (lp + 1) * page > n - window + 1
            assert (table[lp] >= 0) == live, (n, lp)
        m.check()
    assert m.used_pages(0) <= -(-keep // page) + -(-window // page) + 2
    m.close("a")
    assert m.used_pages(0) == 0
    m.check()


def test_layers_that_keep_first_tokens_have_pages_of_their_own():
    spec = [CacheSpec(kv=KVSpec(1, 2, 8, None, None, k)) for k in (0, 4, 4, 5)]
    layout = CacheLayout.build(spec, [None] * 4)
    assert [r.group for r in layout.refs] == [0, 1, 1, 2]


# ---- the plain functions against other formulations -----------------------------------------------------------------
def test_plain_convolution_equals_conv1d():
    torch.manual_seed(1)
    u, w = torch.randn(11, 6, dtype=P.F), torch.randn(6, 4, dtype=P.F)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T[None], (3, 0)), w[:, None], groups=6)[0].T
    assert torch.allclose(P.short_conv(u, w), want, atol=1e-12)


def test_plain_attention_equals_a_masked_softmax_with_a_key_of_score_zero():
    torch.manual_seed(2)
    T, H, G, d, vd = 23, 6, 3, 5, 4
    q, k, v = (torch.randn(T, n, e, dtype=P.F) for n, e in ((H, d), (G, d), (G, vd)))
    kk, vv = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    for size, keep, cap, dist, one in ((7, 0, 2.0, True, True), (4, 3, None, False, False), (None, 0, None, True, True), (5, 9, 3.0, True, False)):
        s = torch.einsum("ihd,jhd->hij", q, kk) * 0.3
        if cap:
            s = torch.tanh(s / cap) * cap
        if dist:
            s = s - torch.pow(torch.tensor(0.5, dtype=P.F), 8 * torch.arange(1, H + 1, dtype=P.F) / H)[:, None, None] * (i - j)
        seen = (j <= i) & (torch.ones_like(i - j, dtype=torch.bool) if size is None else ((j > i - size) | (j < keep)))
        s = s.masked_fill(~seen, -math.inf)
        if one:          # one more key, of score 0 and value 0
            s = torch.cat([s, torch.zeros(H, T, 1, dtype=P.F)], -1)
        p = torch.softmax(s, -1)[..., :T]
        assert torch.allclose(P.attention(q, k, v, 0.3, size, keep, cap, dist, one), torch.einsum("hij,jhe->ihe", p, vv), atol=1e-12)


def test_plain_delta_rule_equals_its_transition_matrices():
    torch.manual_seed(3)
    T, d, e = 9, 4, 3
    q, k, v = torch.randn(T, d, dtype=P.F), P.unit_vector(torch.randn(T, d, dtype=P.F)), torch.randn(T, e, dtype=P.F)
    g, beta = torch.rand(T, dtype=P.F), torch.rand(T, dtype=P.F)
    S = torch.zeros(d, e, dtype=P.F)
    out = []
    for t in range(T):
        S = g[t] * (torch.eye(d, dtype=P.F) - beta[t] * torch.outer(k[t], k[t])) @ S + beta[t] * torch.outer(k[t], v[t])
        out.append(q[t] @ S)
    assert torch.allclose(P.delta_rule(q, k, v, g, beta), torch.stack(out), atol=1e-12)


def test_plain_gated_linear_attention_equals_the_sum_over_earlier_tokens():
    torch.manual_seed(4)
    T, d, e = 10, 4, 3
    q, k, v, a = torch.randn(T, d, dtype=P.F), torch.randn(T, d, dtype=P.F), torch.randn(T, e, dtype=P.F), torch.rand(T, d, dtype=P.F)
    L = torch.cumsum(torch.log(a), 0)
    want = torch.stack([sum(((q[t] * k[s] * torch.exp(L[t] - L[s])).sum()) * v[s] for s in range(t + 1)) for t in range(T)])
    assert torch.allclose(P.gated_linear(q, k, v, a), want, atol=1e-12)


def test_plain_decays():
    torch.manual_seed(5)
    h = torch.randn(7, 6, dtype=P.F)
    W = {"m.a": torch.randn(3, 6, dtype=P.F), "m.dt_bias": torch.randn(3, dtype=P.F), "m.A_log": torch.randn(3, dtype=P.F),
         "m.a1": torch.randn(2, 6, dtype=P.F), "m.a2": torch.randn(8, 2, dtype=P.F), "m.a2.b": torch.randn(8, dtype=P.F)}
    z = h @ W["m.a"].T + W["m.dt_bias"]
    assert torch.allclose(P.head_decay(h, W, "m"), (1 + z.exp()) ** -W["m.A_log"].exp(), atol=1e-12)
    z = h @ W["m.a1"].T @ W["m.a2"].T + W["m.a2.b"]
    assert torch.allclose(P.channel_decay(h, W, "m", 5.0), (1 + (-z).exp()) ** -0.2, atol=1e-12)


def test_plain_rotation_is_a_complex_product_of_neighbours():
    torch.manual_seed(6)
    x = torch.randn(6, 2, 8, dtype=P.F)
    y = P.rotate_pairs(x, {"dims": 8, "base": 100.0})
    f = 100.0 ** (-torch.arange(4, dtype=P.F) / 4)
    z = torch.view_as_complex(x.reshape(6, 2, 4, 2).contiguous()) * torch.polar(torch.ones(6, 4, dtype=P.F), torch.arange(6, dtype=P.F)[:, None] * f)[:, None]
    assert torch.allclose(y, torch.view_as_real(z).reshape(6, 2, 8), atol=1e-12)


def test_plain_passes_of_the_loop():
    """Two passes over a stretch equal a model that has the stretch twice, fed by hand between the two."""
    cfg = config("C")
    cfg["loop"] = {"start": 1, "stop": 2, "times": 2}
    W = random_weights(cfg, 3)
    toks = [5, 9, 1, 22]
    logits, streams = P.forward(toks, cfg, W)
    assert streams.shape[0] == len(cfg["layers"]) + 1
    Wd = {k: v.double() for k, v in W.items()}
    x0 = Wd["embed"][toks] * cfg["embedding"]["scale"]
    x = streams[1] + x0 + Wd["loop.step"][1]
    h = P.layer_norm1p(x, Wd["l1.norm1"], cfg["norm"]["eps"])
    x = x + P.parallel_2(h, Wd, "l1.mix", cfg["layers"][1]["mixer"], cfg["norm"]["eps"])
    x = x + P.dense(P.layer_norm1p(x, Wd["l1.norm2"], cfg["norm"]["eps"]), Wd, "l1.mlp")
    assert torch.allclose(x, streams[2], atol=1e-10)
