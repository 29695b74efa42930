"""Laralix on the GPU: every new kernel alone against the plain functions, then the model through the engine's own step
function, cache manager, scheduler and replay tool against the plain implementation, on five tiny configurations and on
configurations drawn at random."""
import random

import numpy as np
import pytest
import torch

from lightllm_b200 import Engine, EngineCore, EngineOptions, StepEntry
from lightllm_b200.csrc import ops
from lightllm_b200.parts import linear as L
from tests.laralix_configs import CONFIGS, PAGE_SIZE, config, random_config, random_weights, write_model
from tests.plain import laralix_plain as P
from tests.tolerances import FLOAT32_ATOL, LARALIX_BF16_WORST_REL, logits_std, record
from tests.trace_util import Trace, compare_with_plain, run_trace

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
NAN = float("nan")


def dev(t, dtype=None):
    return t.to(DEV, dtype=dtype).contiguous()


def i32(xs):
    return dev(torch.tensor(list(xs), dtype=torch.int32))


def close(got, want, dtype, what, rel=None):
    """float32: 2e-5 of the result's scale; bfloat16: a few roundings of 2^-9."""
    scale = float(want.abs().max()) + 1e-6
    tol = (2e-5 if dtype == "float32" else 1.5e-2) * scale if rel is None else rel * scale
    err = float((got.double().cpu() - want.double()).abs().max())
    assert err <= tol, f"{what}: max |diff| {err:.3e} > {tol:.3e}"


def spans_of(parts):
    """Device arrays (span_row, span_len, span_pos, span_slot, count) for parts (request, slot, from, to)."""
    starts = np.cumsum([0] + [b - a for _, _, a, b in parts])[:-1]
    return (i32(starts), i32(b - a for _, _, a, b in parts), i32(a for _, _, a, _ in parts), i32(s for _, s, _, _ in parts),
            len(parts))


def pieces_of(parts, chunk):
    counts = [-(-(b - a) // chunk) for _, _, a, b in parts]
    span = [s for s, c in enumerate(counts) for _ in range(c)]
    num = [j for c in counts for j in range(c)]
    first = np.cumsum([0] + counts)[:-1]
    return i32(span), i32(num), i32(first), len(span), chunk


# ---------------------------------------------------------------------------------------------------------------------
# attention: the bias by distance, kept first tokens
# ---------------------------------------------------------------------------------------------------------------------
class Mask:
    """What one attention case switches on."""

    def __init__(self, window, keep=0, cap=None, bias=False, one=False):
        self.window, self.keep, self.cap, self.bias, self.one = window, keep, cap, bias, one

    def plain(self, q, k, v, start, scale, **edit):
        a = {**vars(self), **edit}
        return P.attention(q.double(), k.double(), v.double(), scale, a["window"], a["keep"], a["cap"], a["bias"], a["one"], start)

    def kernel(self, H):
        return dict(softcap=self.cap or 0.0, keep=self.keep, sinks=torch.zeros(H, device=DEV) if self.one else None,
                    slopes=dev(torch.tensor(P.slopes(H), dtype=torch.float32)) if self.bias else None)


def paged(k, v, page, start, mask, dtype, seed):
    """The caches and block table of one request that holds ``len(k)`` tokens and whose next rows begin at ``start``: pages that
    no row sees any more are given back (-1 in the table), and every row of the pool that the request does not hold is NaN."""
    n = k.shape[0]
    pages = torch.randperm(96, generator=torch.Generator().manual_seed(seed))[: -(-n // page)].to(torch.int32)
    lo = max(0, start - mask.window + 1) if mask.window else 0
    bt = torch.full((1, len(pages) + 1), -1, dtype=torch.int32)
    kc = torch.full((96 * page, *k.shape[1:]), NAN, dtype=DT[dtype])
    vc = torch.full((96 * page, *v.shape[1:]), NAN, dtype=DT[dtype])
    for j, pg in enumerate(pages.tolist()):
        a, b = j * page, min(n, (j + 1) * page)
        if b > lo or a < mask.keep:
            bt[0, j] = pg
            kc[pg * page: pg * page + b - a], vc[pg * page: pg * page + b - a] = k[a:b], v[a:b]
    return dev(kc), dev(vc), dev(bt)


def made_query(q, k, last, mask):
    """The last row's last head (the one with the smallest slope) matches the keys just inside and just outside the window and
    the last kept and first not kept token alike; under a sink the first head has scores of 0 before the bias."""
    if mask.one:
        q[-1, 0] = 0.0
    at = [p for p in ((last - mask.window + 1, last - mask.window) if mask.window else ()) if p >= 0]
    at += [p for p in ((mask.keep - 1, mask.keep) if mask.keep else ()) if 0 <= p <= last]
    if at:
        for p in set(at):          # (keys of full length among short ones)
            k[p, -1] *= k.shape[-1] ** 0.5 / float(k[p, -1].float().norm())
        slope = P.slopes(q.shape[1])[-1] if mask.bias and not mask.cap else 0.0          # scores of about 6 after the bias
        q[-1, -1] = sum(k[p, -1].float() * (1 + slope * (last - p) / 6) for p in set(at)).to(q.dtype)
    return at


def worth(mask, want, q, k, v, start, scale, least=0.04):
    """Every mechanism of the case moves the result by far more than the tolerance."""
    edits = []
    last = start + q.shape[0] - 1
    if mask.window and last - mask.window >= max(mask.keep, 0):
        edits.append({"window": mask.window + 1})
        if mask.window > 1 and last - mask.window + 1 >= mask.keep:
            edits.append({"window": mask.window - 1})
    if mask.keep and mask.window and last - mask.window >= mask.keep:
        edits += [{"keep": mask.keep - 1}, {"keep": mask.keep + 1}]
    if mask.bias and last > 4:
        edits.append({"bias": False})
    if mask.one:
        edits.append({"one": False})
    for e in edits:
        other = mask.plain(q[-1:], k, v, last, scale, **e)
        moved = (other[0] - want[-1]).abs().amax(-1) / want[-1].abs().amax(-1)          # of every head's own result
        assert float(moved.max()) > least, e


MASKS = [Mask(23, 0, 4.0, True, True), Mask(9, 5, None, False, False), Mask(40, 16, None, True, False), Mask(None, 0, 6.0, True, True),
         Mask(1, 3, None, False, True), Mask(30, 70, 5.0, True, False)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,vd", [(4, 2, 12, 20), (3, 3, 9, 7), (6, 1, 18, 18), (20, 4, 64, 64), (2, 1, 34, 48)])
@pytest.mark.parametrize("mask", MASKS, ids=lambda m: "-".join(str(x) for x in vars(m).values()))
def test_cuda_core_attention(mask, dtype, H, G, d, vd):
    torch.manual_seed(H * d)
    page, n = 8, 170
    k, v = (0.3 * torch.randn(n, G, d)).to(DT[dtype]), torch.randn(n, G, vd).to(DT[dtype])
    scale = (1.5 * mask.cap if mask.cap else 6.0) / d
    from lightllm_b200.parts.attention import AttentionMixer
    part = AttentionMixer("m", 32, H, G, d, v_head_dim=vd)
    for start, rows, bq, nsplit in ((120, 50, part.tile_height(), 1), (120, 20, 1, 3), (0, 30, part.tile_height(), 1),
                                    (n - 1, 1, 1, 1), (n - 1, 1, 1, 4), (7, 2, 2, 1)):
        q = (torch.randn(rows, H, d) * 0.5).to(DT[dtype])
        made_query(q, k, start + rows - 1, mask)
        kc, vc, bt = paged(k[: start + rows], v[: start + rows], page, start, mask, dtype, rows)
        want = mask.plain(q, k, v, start, scale)
        out = torch.full((rows, H * vd), NAN, dtype=DT[dtype], device=DEV)
        tq0 = list(range(0, rows, bq))
        scratch = torch.empty(ops.attention_scratch_floats(len(tq0), H, vd, bq, nsplit), device=DEV) if nsplit > 1 else None
        ops.paged_attention_simt(dev(q).view(rows, H * d), kc, vc, out, i32([0] * len(tq0)), i32(tq0), len(tq0), i32([0]),
                                 i32([rows]), i32([start]), bt, bt.shape[1], page, H, G, d, mask.window or 0, scale, bq, nsplit,
                                 scratch, v_head_dim=vd, **mask.kernel(H))
        close(out.view(rows, H, vd), want, dtype, f"start {start}, {rows} rows, bq {bq}, {nsplit} pieces")
        if start > 100 and dtype == "float32":          # (the same kernel in both; narrow heads leave little room above bfloat16's rounding)
            worth(mask, want, q, k, v, start, scale, least=0.005)


TC_MASKS = [Mask(150, 0, 8.0, True, True), Mask(130, 20, None, False, False), Mask(16, 140, None, False, False), Mask(200, 300, 8.0, True, True),
            Mask(None, 0, None, True, False), Mask(1, 4, None, False, True), Mask(64, 128, None, True, False), Mask(129, 1, 5.0, False, False)]


@pytest.mark.parametrize("H,G,hd", [(4, 2, 64), (4, 1, 128), (16, 1, 64), (3, 3, 128)])
@pytest.mark.parametrize("mask", TC_MASKS, ids=lambda m: "-".join(str(x) for x in vars(m).values()))
def test_tensor_core_attention(mask, H, G, hd):
    """The tcgen05 kernel (portions, key ranges whole and cut into pieces that cross from the kept tokens' tiles into the
    window's) and the decode kernel (pieces merged in a cluster and through scratch)."""
    from lightllm_b200.engine.batch import Span, StepContext
    torch.manual_seed(H + hd)
    page, n = 16, 700
    k, v = (0.3 * torch.randn(n, G, hd)).to(torch.bfloat16), torch.randn(n, G, hd).to(torch.bfloat16)
    scale = (1.5 * mask.cap if mask.cap else 6.0) / hd
    for start, rows, pieces in ((0, 140, None), (380, 130, 2), (690, 10, None), (555, 45, 1), (3, 2, None), (127, 3, 1)):
        q = (torch.randn(rows, H, hd) * 0.5).to(torch.bfloat16)
        made_query(q, k, start + rows - 1, mask)
        kc, vc, bt = paged(k[: start + rows], v[: start + rows], page, start, mask, "bfloat16", rows)
        out = torch.full((rows, H * hd), NAN, dtype=torch.bfloat16, device=DEV)
        ctx = StepContext()
        ctx.spans, ctx.device = [Span("a", 0, start, rows, 0)], DEV
        ctx.iota, ctx.zeros = i32([0]), i32([0])
        ts, tq, nt, cut = ctx.attention_items(1, mask.window or 0, pieces, H, 296, keep=mask.keep)
        ops.paged_attention_tcgen05(dev(q).view(rows, H * hd), kc, vc, out, ts, tq, nt, i32([0]), i32([rows]), i32([start]),
                                    bt, bt.shape[1], page, H, G, hd, mask.window or 0, scale, cut=cut, **mask.kernel(H))
        ops.check_async_errors(DEV)
        want = mask.plain(q, k, v, start, scale)
        close(out.view(rows, H, hd), want, "bfloat16", f"tcgen05, start {start}, {rows} rows, pieces of {pieces}")
        if start > 100:
            worth(mask, want, q, k, v, start, scale)
    for pos in (n - 1, 330, 130, 0):
        for nsplit in (1, 4, 20):
            q = (torch.randn(1, H, hd) * 0.5).to(torch.bfloat16)
            made_query(q, k, pos, mask)
            kc, vc, bt = paged(k[: pos + 1], v[: pos + 1], page, pos, mask, "bfloat16", pos)
            out = torch.full((1, H * hd), NAN, dtype=torch.bfloat16, device=DEV)
            scratch = None
            if nsplit > ops.decode_mma_cluster_splits():
                scratch = torch.empty(ops.attention_scratch_floats(1, H, hd, 1, nsplit), device=DEV)
            ops.paged_decode_mma(dev(q).view(1, H * hd), kc, vc, out, i32([0]), i32([0]), 1, i32([0]), i32([pos]), bt,
                                 bt.shape[1], page, H, G, hd, mask.window or 0, scale, nsplit, scratch, **mask.kernel(H))
            want = mask.plain(q, k, v, pos, scale)
            close(out.view(1, H, hd), want, "bfloat16", f"decode at {pos}, {nsplit} pieces")
            if pos > 300:
                worth(mask, want, q, k, v, pos, scale)


def test_a_bias_that_outweighs_the_scores_leaves_nothing_lost():
    """Slopes near one and scores that favour far keys by more than float exponents hold beside the near ones: the shift by the
    bound must follow the bias."""
    from lightllm_b200.engine.batch import Span, StepContext
    torch.manual_seed(0)
    H, hd, n, page = 64, 64, 400, 16
    mask = Mask(None, 0, None, True, False)
    k, v = torch.randn(n, 64, hd).to(torch.bfloat16), torch.randn(n, 64, hd).to(torch.bfloat16)
    q = torch.zeros(200, H, hd)
    for r in range(200):          # every row dislikes its own key by 60 and likes the key 100 positions before by 60
        q[r] = k[100 + r].float() - k[200 + r].float()
    q = q.to(torch.bfloat16)
    kc, vc, bt = paged(k, v, page, 200, mask, "bfloat16", 1)
    out = torch.full((200, H * hd), NAN, dtype=torch.bfloat16, device=DEV)
    ctx = StepContext()
    ctx.spans, ctx.device = [Span("a", 0, 200, 200, 0)], DEV
    ctx.iota, ctx.zeros = i32([0]), i32([0])
    ts, tq, nt, cut = ctx.attention_items(1, 0, None, H, 296)
    ops.paged_attention_tcgen05(dev(q).view(200, H * hd), kc, vc, out, ts, tq, nt, i32([0]), i32([200]), i32([200]), bt, bt.shape[1],
                                page, H, 64, hd, 0, 1.0, cut=cut, **mask.kernel(H))
    ops.check_async_errors(DEV)
    close(out.view(200, H, hd)[::10], torch.cat([mask.plain(q[r:r + 1], k, v, 200 + r, 1.0) for r in range(0, 200, 10)]), "bfloat16", "steep bias", rel=3e-2)


# ---------------------------------------------------------------------------------------------------------------------
# recurrences
# ---------------------------------------------------------------------------------------------------------------------
SPAN_STEPS = [[("a", 2, 0, 90), ("c", 0, 0, 18)],                 # c ends here; its slot 0 is used again by b
              [("a", 2, 90, 91), ("b", 0, 0, 1)],
              [("b", 0, 1, 3), ("a", 2, 91, 92)],
              [("a", 2, 92, 93), ("b", 0, 3, 4)],
              [("b", 0, 4, 110), ("a", 2, 93, 230)]]
SPAN_LENS = {"a": 230, "b": 110, "c": 18}


@pytest.mark.parametrize("H,G,d,vd", [(4, 2, 6, 10), (2, 1, 11, 5), (6, 2, 72, 9), (2, 2, 32, 64), (3, 1, 64, 16), (1, 1, 8, 8), (2, 1, 130, 24)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_delta_rule_with_one_decay_a_head(dtype, H, G, d, vd):
    """Spans that begin, continue, use a slot again and single tokens; in blocks of tokens and token by token; the state lies
    behind other floats of its slot; a stretch that forgets at once."""
    torch.manual_seed(H * d + vd)
    unit = lambda x: x / x.norm(dim=-1, keepdim=True)
    data, want = {}, {}
    bias, A = torch.randn(H) - 2.0, torch.randn(H) - 0.5
    for r, n in SPAN_LENS.items():
        q, k = unit(torch.randn(n, G, d)), unit(torch.randn(n, G, d))
        v, gates = torch.randn(n, H, vd), torch.randn(n, 2 * H + 3).to(DT[dtype])
        if r == "a":
            gates[40:60, H + 1: 2 * H + 1] = 9.0
        data[r] = (q, k, v, gates)
        g = torch.exp(-torch.exp(A.double()) * torch.nn.functional.softplus(gates[:, H + 1: 2 * H + 1].double() + bias.double()))
        beta = torch.sigmoid(gates[:, 1: H + 1].double())
        want[r] = torch.stack([P.delta_rule(q[:, h // (H // G)].double(), k[:, h // (H // G)].double(), v[:, h].double(), g[:, h],
                                            beta[:, h]) for h in range(H)], 1)
    off, size = 5, H * d * vd
    for blocked in (False, True):
        state = torch.full((4, off + size + 7), NAN, device=DEV)
        for parts in SPAN_STEPS:
            q, k, v, gates = (dev(torch.cat([data[r][i][a:b] for r, _, a, b in parts])) for i in range(4))
            T = q.shape[0]
            out = torch.full((T, H * vd), NAN, device=DEV)
            ops.delta_rule(q.view(T, -1), k.view(T, -1), v.view(T, -1), None, gates[:, 1: H + 1], spans_of(parts), H, G, d, vd, state,
                           off, out, blocked=blocked, head_decay=(gates[:, H + 1: 2 * H + 1], dev(bias), dev(torch.exp(A))))
            at = 0
            for r, _, a, b in parts:
                close(out[at:at + b - a].view(b - a, H, vd), want[r][a:b], "float32", f"{r}[{a}:{b}] blocked={blocked}", rel=4e-5)
                at += b - a
        assert torch.isnan(state[2, :off]).all() and torch.isnan(state[2, off + size:]).all() and torch.isnan(state[1]).all()
        assert torch.isfinite(state[2, off: off + size]).all()


@pytest.mark.parametrize("H,d,vd", [(3, 10, 7), (1, 8, 8), (2, 130, 12), (4, 16, 32), (2, 64, 72), (1, 96, 40), (2, 300, 5), (3, 24, 300)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gated_linear_attention_over_spans_pieces_and_slots(dtype, H, d, vd):
    """As above, the spans whole and in pieces that run side by side.  The inputs are what the kernel reads, so the result is
    judged as float32 in both precisions."""
    torch.manual_seed(H * d + vd)
    C = 2 * H * d + H * vd + 5
    data, want = {}, {}
    for r, n in SPAN_LENS.items():
        src = (torch.randn(n, C) * 0.5).to(DT[dtype])
        g = -torch.nn.functional.softplus(torch.randn(n, H * d)) / 8
        if r == "a":
            g[30:45] = -40.0                          # forgets at once
        data[r] = (src, g)
        x, al = src.double(), torch.exp(g.double()).view(n, H, d)
        q, k = x[:, 2: 2 + H * d].reshape(n, H, d) * 0.3, x[:, 2 + H * d: 2 + 2 * H * d].reshape(n, H, d)
        v = x[:, 2 + 2 * H * d: 2 + 2 * H * d + H * vd].reshape(n, H, vd)
        want[r] = torch.stack([P.gated_linear(q[:, h], k[:, h], v[:, h], al[:, h]) for h in range(H)], 1)
    off, size = 3, H * d * vd
    for chunk in (None, 16, 33, 64):
        state = torch.full((4, off + size + 2), NAN, device=DEV)
        for parts in SPAN_STEPS:
            src, g = (dev(torch.cat([data[r][i][a:b] for r, _, a, b in parts])) for i in range(2))
            out = torch.full((src.shape[0], H * vd), NAN, device=DEV)
            ops.gated_linear(src, 2, 2 + H * d, 2 + 2 * H * d, g, 0.3, spans_of(parts), H, d, vd, state, off, out,
                             pieces=None if chunk is None else pieces_of(parts, chunk))
            at = 0
            for r, _, a, b in parts:
                close(out[at:at + b - a].view(b - a, H, vd), want[r][a:b], "float32", f"{r}[{a}:{b}] pieces of {chunk}", rel=4e-5)
                at += b - a
        assert torch.isnan(state[2, :off]).all() and torch.isnan(state[2, off + size:]).all() and torch.isnan(state[1]).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,R,N", [(1, 3, 30), (16, 16, 64), (17, 1, 8), (70, 20, 260)])
def test_log_sigmoid_decays_from_a_low_rank_pair(dtype, T, R, N):
    torch.manual_seed(T + N)
    x, w, b = torch.randn(T, R + 4).to(DT[dtype]), torch.randn(N, R).to(DT[dtype]), torch.randn(N) * 3
    b[0], b[-1] = 60.0, -60.0                        # saturated both ways
    out = torch.empty(T, N, device=DEV)
    ops.low_rank_up(dev(x), 2, dev(w), out, bias=dev(b), mode="log_sigmoid", multiplier=1 / 5.0)
    z = x[:, 2: 2 + R].double() @ w.double().T + b.double()
    want = torch.nn.functional.logsigmoid(z) / 5.0
    assert float(((out.double().cpu() - want).abs() / (want.abs() + 1e-12)).max()) < 1e-4


# ---------------------------------------------------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("n,T,D", [(2, 1, 44), (2, 37, 256), (1, 5, 50), (4, 9, 1030), (3, 300, 64), (2, 40, 1028), (4, 3, 2048), (2, 5, 2052), (2, 7, 896)])
def test_normed_branches_join_in_one_pass(n, T, D):
    torch.manual_seed(D)
    x, w, dst = torch.randn(n, T, D) * 3, torch.randn(n, D), torch.randn(T, D)
    out = dev(dst)
    ops.rmsnorm_sum(dev(x), dev(w), 1e-5, out)
    close(out, dst.double() + sum(P.rms_norm(x[i].double(), w[i].double(), 1e-5) for i in range(n)), "float32", "sum of normed branches")


def test_the_embedding_and_a_step_vector_join_the_stream():
    torch.manual_seed(0)
    x, e, v = torch.randn(7, 50), torch.randn(7, 50), torch.randn(50)
    out = dev(x)
    ops.add_sum_row(out, dev(e), dev(v))
    assert torch.equal(out.cpu(), (x + e) + v)
    table = torch.randn(20, 50).to(torch.bfloat16)
    ids = [3, 0, 19]
    stream, copy = torch.empty(3, 50, device=DEV), torch.empty(3, 50, device=DEV)
    ops.embedding(i32(ids), dev(table), stream, scale=3.3, copy=copy)          # a float copy of a bfloat16 table's rows
    assert torch.equal(stream, copy)
    close(stream, table[ids].double() * 3.3, "float32", "scaled embedding", rel=1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,N,K", [(1, 96, 64), (5, 44, 28), (40, 301, 128), (64, 256, 1024), (100, 130, 72), (200, 512, 256), (700, 1536, 192),
                                   (300, 128, 4096)])
def test_contractions_with_a_scale_on_the_outputs(dtype, M, N, K):
    """Both float epilogues, with few rows, up to 128, many, and K cut into pieces; the unscaled call is not touched."""
    torch.manual_seed(M + N)
    x, w, b = torch.randn(M, K).to(DT[dtype]), (torch.randn(N, K) / K ** 0.5).to(DT[dtype]), torch.randn(N)
    res = torch.randn(M, N)
    y = x.double() @ w.double().T
    for bias in (None, b):
        full = y if bias is None else y + b.double()
        close(L.linear(dev(x), dev(w), None if bias is None else dev(b), L.STORE_F32, scale=-1.7), -1.7 * full, "float32", "store", rel=3e-5)
        for scale in (0.6, 1.0):
            got = dev(res)
            L.linear(dev(x), dev(w), None if bias is None else dev(b), L.RESIDUAL, residual=got, scale=scale)
            close(got, res.double() + scale * full, "float32", f"residual {scale}", rel=3e-5)
    ops.check_async_errors(DEV)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,G,d", [(5, 4, 2, 12), (1, 1, 1, 8), (300, 8, 2, 64), (9, 18, 1, 10)])
def test_whole_projection_norm_beside_values_that_are_the_keys_as_projected(dtype, T, H, G, d):
    torch.manual_seed(T)
    src = torch.randn(T, 3 + (H + G) * d + 2).to(DT[dtype])
    wq, wk = 1 + 0.2 * torch.randn(H * d), 1 + 0.2 * torch.randn(G * d)
    slots = torch.randperm(T + 4)[:T].tolist()
    k, v = (torch.full((T + 4, G, d), NAN, device=DEV, dtype=DT[dtype]) for _ in range(2))
    q = torch.empty(T, H * d, device=DEV, dtype=DT[dtype])
    ops.qkv_prepare(dev(src), 3, 3 + H * d, 3 + H * d, H, G, d, d, i32(range(T)), i32(slots), q, k, v, dev(wq), dev(wk), 1e-5)
    x = src.double()
    close(q, P.rms_norm(x[:, 3: 3 + H * d], wq.double(), 1e-5), dtype, "q", rel=None if dtype == "float32" else 5e-3)
    keys = x[:, 3 + H * d: 3 + (H + G) * d]
    close(k[slots].view(T, -1), P.rms_norm(keys, wk.double(), 1e-5), dtype, "k", rel=None if dtype == "float32" else 5e-3)
    assert torch.equal(v[slots].view(T, -1).cpu(), src[:, 3 + H * d: 3 + (H + G) * d])


# ---------------------------------------------------------------------------------------------------------------------
# the model through the engine
# ---------------------------------------------------------------------------------------------------------------------
def make_model(tmp_path, name, dtype, seed=3, sharp=1.0, edit=None, cfg=None):
    cfg = config(name) if cfg is None else cfg
    for layer in cfg["layers"]:
        layer["mixer"].get("left", layer["mixer"])["scale"] *= sharp
    w = random_weights(cfg, seed, store=DT[dtype])
    if edit is not None:
        edit(cfg, w)
    return write_model(cfg, w, str(tmp_path / f"lar_{name}_{seed}_{dtype}")), cfg, w


def core_for(d, dtype, name, pages=64, max_seqs=4, max_tokens=1024, graphs=True):
    return EngineCore(d, EngineOptions(dtype=dtype, max_seq_len=max_tokens, max_batch_tokens=max_tokens,
                                       page_size=PAGE_SIZE.get(name, 16), num_pages=pages, max_seqs=max_seqs, use_cuda_graphs=graphs))


def plain_logits(toks, w, cfg):
    return P.forward(toks, cfg, w)[0].float()


def atol_for(name, dtype, plain):
    """float32: the largest difference of any logit, 1e-4 on logits of order one.  bfloat16: the root mean square over a
    row of logits (mean taken off), at most twice the worst that a recorded run showed, relative to the logits' spread."""
    std = logits_std(plain)
    return (FLOAT32_ATOL * max(1.0, std)) if dtype == "float32" else 2.0 * LARALIX_BF16_WORST_REL[name] * std


def error(got, plain, dtype) -> float:
    d = (got.double() - plain.double())
    if dtype == "float32":
        return float(d.abs().max())
    return float((d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt().max())


LENGTHS = {"A": [1, 2, 17, 33, 70, 130, 64, 49], "B": [3, 40, 131, 290, 129, 64], "C": [1, 5, 40, 90, 33, 64, 17],
           "D": [1, 3, 20, 45, 16, 70, 33, 9], "E": [2, 50, 140, 127, 64]}


def build_trace(name, cfg, seed=11):
    rng = random.Random(seed)
    seqs = {f"r{i}": [rng.randrange(cfg["vocab"]) for _ in range(n)] for i, n in enumerate(LENGTHS[name])}
    tr = Trace({f"{regime}{rid}": toks for rid, toks in seqs.items() for regime in "wtpm"})
    for rid in seqs:
        tr.whole(f"w{rid}")
    for rid, toks in seqs.items():
        if len(toks) > 2:
            tr.last_one_by_one(f"t{rid}", tail=40)
    for i, rid in enumerate(seqs):
        if len(seqs[rid]) > 1:
            tr.portions(f"p{rid}", [[16, 7, 2, 5, 3, 2], [2, 2, 9, 31, 4], [13, 2, 64, 3], [200, 33, 2, 129]][i % 4])
    prompt_len = {f"m{rid}": max(2, len(toks) - 12) if len(toks) > 14 else len(toks) for rid, toks in seqs.items()}
    tr.mixed([f"m{rid}" for rid in seqs], prompt_len, seed=5, sizes=(2, 3, 7, 16, 40, 130) if name in "BE" else (2, 3, 5, 7, 16))
    return tr, seqs


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_all_regimes(name, dtype, tmp_path):
    """Through bin/trace_run: whole prompts, the last tokens one by one, portions down to two tokens, and up to four
    live requests mixed in a pool so small that pages and state slots are used again."""
    d, cfg, w = make_model(tmp_path, name, dtype)
    tr, seqs = build_trace(name, cfg)
    once = {rid: plain_logits(toks, w, cfg) for rid, toks in seqs.items()}
    plain = {f"{regime}{rid}": lg for rid, lg in once.items() for regime in "wtpm"}
    got = run_trace(d, dtype, tr, str(tmp_path / "out"), ["--page-size", str(PAGE_SIZE[name])])
    worst = compare_with_plain(tr, got, plain, atol_for(name, dtype, once), f"Laralix {name} {dtype}", rms=dtype != "float32")
    record(f"replay Laralix {name} {dtype} ({len(tr.steps)} steps, pool for {tr.max_tokens} tokens)", worst, logits_std(once))


def stepwise(core, rid, toks, cuts):
    """Feed ``toks`` in portions of the given sizes (the rest one by one); returns logits of every position."""
    core.open(rid)
    rows, at, i = [], 0, 0
    while at < len(toks):
        c = min(cuts[i], len(toks) - at) if i < len(cuts) else 1
        rows.append(core.step([StepEntry(rid, toks[at:at + c], list(range(c)))]).float().cpu())
        at += c
        i += 1
    core.close(rid)
    return torch.cat(rows)


def only_attention(cfg, w):
    """The attention alone decides: the recurrences' and the feed-forwards' last projections are zero."""
    for k in w:
        if k.endswith("right.o") or k.endswith("mlp.down"):
            w[k] = torch.zeros_like(w[k])


def edited(cfg, key, by):
    """The configuration with every window (or number of kept tokens) changed by one."""
    out = {**cfg, "layers": [dict(l, mixer=dict(l["mixer"])) for l in cfg["layers"]]}
    for layer in out["layers"]:
        left = layer["mixer"].get("left") or {}
        if key in (left.get("mask") or {}):
            layer["mixer"]["left"] = dict(left, mask=dict(left["mask"], **{key: left["mask"][key] + by}))
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "D", "E"])
def test_sharp_attention_at_window_edges_and_kept_tokens(tmp_path, name, dtype):
    """The attention's scale multiplied and every other path into the stream silenced, so that single keys carry a row's output:
    the prompt in portions that end inside pages, then tokens one by one, so that windows pass over decoded tokens and over the
    kept ones.  The plain implementation itself, with every window or every number of kept tokens one off, lies far outside
    the bound."""
    d, cfg, w = make_model(tmp_path, name, dtype, seed=8, sharp=2.5, edit=only_attention)
    rng = random.Random(2)
    toks = [rng.randrange(cfg["vocab"]) for _ in range({"B": 300, "E": 200}.get(name, 140))]
    plain = plain_logits(toks, w, cfg)
    core = core_for(d, dtype, name)
    got = stepwise(core, "a", toks, [129, 2, 31, 2] if name in "BE" else [9, 2, 16, 38, 2, 13])
    err = error(got, plain, dtype)
    record(f"sharp Laralix {name} {dtype}", err, logits_std(plain))
    tol = atol_for(name + " sharp", dtype, plain)
    assert err <= tol
    core.runner.check_device_errors()
    for key, by in (("size", -1), ("size", 1), ("keep_first", -1), ("keep_first", 1)):
        assert error(plain_logits(toks, w, edited(cfg, key, by)), plain, dtype) > 1.5 * tol, (key, by)


def only_recurrence(cfg, w):
    """The recurrences alone decide, and they forget slowly."""
    for k in w:
        if k.endswith("left.o") or k.endswith("mix.o") or k.endswith("mlp.down"):
            w[k] = torch.zeros_like(w[k])
        elif k.endswith("A_log"):
            w[k] = torch.full_like(w[k], -4.0)
        elif k.endswith("a2.b"):
            w[k] = torch.full_like(w[k], 5.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "D", "E"])
def test_a_lost_state_shows(tmp_path, name, dtype):
    """With recurrences that forget slowly as the stream's only input, the first tokens still weigh at the end: the engine in
    portions and single tokens agrees with the plain implementation, which itself differs widely when the first ten tokens
    are taken away."""
    d, cfg, w = make_model(tmp_path, name, dtype, seed=9, edit=only_recurrence)
    rng = random.Random(3)
    toks = [rng.randrange(cfg["vocab"]) for _ in range(150)]
    plain = plain_logits(toks, w, cfg)
    core = core_for(d, dtype, name)
    got = stepwise(core, "a", toks, [40, 2, 33, 50])
    err = error(got, plain, dtype)
    record(f"recurrence Laralix {name} {dtype}", err, logits_std(plain))
    tol = atol_for(name + " recurrence", dtype, plain)
    assert err <= tol
    off = error(plain_logits(toks[10:], w, cfg)[-20:], plain[-20:], dtype)
    assert off > 1.5 * tol, (off, tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_equals_token_by_token_and_long_decoding(tmp_path, name, dtype):
    """A whole prompt in one step against the same tokens one by one from the first (states and tails are carried through every
    step, windows pass over decoded tokens, pages are given back and taken, kept ones are not)."""
    d, cfg, w = make_model(tmp_path, name, dtype, seed=5)
    rng = random.Random(4)
    toks = [rng.randrange(cfg["vocab"]) for _ in range(220)]
    plain = plain_logits(toks, w, cfg)
    core = core_for(d, dtype, name)
    whole = stepwise(core, "a", toks, [220])
    one = stepwise(core, "b", toks, [])
    tol = atol_for(name, dtype, plain)
    record(f"Laralix {name} {dtype} token by token", max(error(one, plain, dtype), error(whole, plain, dtype)), logits_std(plain))
    assert error(whole, plain, dtype) <= tol and error(one, plain, dtype) <= tol
    core.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "D", "E"])
def test_a_batch_of_unequal_requests_equals_each_alone_and_slots_are_used_again(tmp_path, name, dtype):
    d, cfg, w = make_model(tmp_path, name, dtype, seed=6)
    rng = random.Random(7)
    toks = {r: [rng.randrange(cfg["vocab"]) for _ in range(n)] for r, n in (("a", 75), ("b", 140), ("c", 9), ("d", 33), ("e", 52))}
    core = core_for(d, dtype, name, max_seqs=3)
    alone = {r: stepwise(core, r, t, [len(t) - 3]) for r, t in toks.items()}
    got = {r: [] for r in toks}

    def step(*feeds, end=()):
        entries = []
        for r, c in feeds:
            if not core.is_open(r):
                core.open(r)
            at = sum(x.shape[0] for x in got[r])
            entries.append(StepEntry(r, toks[r][at:at + c], list(range(c))))
        out = core.step(entries).float().cpu()
        at = 0
        for r, c in feeds:
            got[r].append(out[at:at + c])
            at += c
        for r in end:
            core.close(r)

    # a decodes while b and c bring portions; c ends and d takes its slot in the next step; then e takes a's
    step(("a", 70))
    step(("a", 1), ("b", 100), ("c", 7))
    step(("c", 2), ("a", 1), ("b", 2), end=["c"])
    step(("b", 37), ("d", 33), ("a", 1), end=["d"])
    step(("a", 1), ("b", 1))
    step(("a", 1), end=["a", "b"])
    step(("e", 50))
    step(("e", 2), end=["e"])
    core.cache.check()
    assert core.cache.free_slots == 3
    plain = {r: plain_logits(t, w, cfg) for r, t in toks.items()}
    tol = atol_for(name, dtype, plain)
    worst = 0.0
    for r in toks:
        both = torch.cat(got[r])
        worst = max(worst, error(both, plain[r], dtype))
        assert error(both, plain[r], dtype) <= tol, r
        # the batch and the request alone: float32 differs by the order of split sums only
        assert error(both, alone[r], dtype) <= (3e-5 * max(1.0, logits_std(plain)) if dtype == "float32" else tol), r
    record(f"Laralix {name} {dtype} batch", worst, logits_std(plain))
    core.runner.check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tensor_core", [False, True])
def test_random_configurations_through_the_engine(tmp_path, dtype, tensor_core):
    for seed in range(6):
        cfg = random_config(random.Random(100 * seed + 7 * tensor_core), tensor_core)
        d, cfg, w = make_model(tmp_path, f"random{seed}", dtype, seed=seed, cfg=cfg)
        rng = random.Random(seed)
        toks = [rng.randrange(cfg["vocab"]) for _ in range(rng.choice([60, 120, 150]))]
        plain = plain_logits(toks, w, cfg)
        core = core_for(d, dtype, "random")
        got = stepwise(core, "a", toks, [rng.choice([2, 17, 33, 50]) for _ in range(3)])
        err = error(got, plain, dtype)
        record(f"random Laralix {seed} {dtype} (tensor-core sizes: {tensor_core})", err, logits_std(plain))
        assert err <= atol_for("random", dtype, plain), (seed, cfg)
        core.runner.check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_greedy_generation_through_the_entry_point(tmp_path, name, dtype):
    d, cfg, w = make_model(tmp_path, name, dtype, seed=10)
    rng = random.Random(1)
    prompts = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (1, 9, 70, 23, 41)]
    eng = Engine(d, dtype=dtype, max_seq_len=160, max_batch_tokens=48, page_size=PAGE_SIZE[name], num_pages=40,
                 max_seqs=3, chunk_size=16)
    outs, why = eng.generate(prompts, max_new_tokens=10, temperature=0.0, eos_token_id=-1, return_reasons=True)
    assert why == ["length"] * 5 and all(len(o) == 10 for o in outs)
    margin_rel = 3e-4 if dtype == "float32" else 3.0 * LARALIX_BF16_WORST_REL[name]
    for p, o in zip(prompts, outs):
        lg = plain_logits(list(p) + o, w, cfg)
        for i, tok in enumerate(o):          # each token is the plain argmax given the same history
            row = lg[len(p) - 1 + i]
            top = torch.topk(row, 2).values
            assert tok == int(torch.argmax(row)) or float(row.max() - row[tok]) < margin_rel * float(row.std()), (p, o, i, top)
    eng.core.cache.check()
    assert eng.core.cache.free_slots == 3
    eng.core.runner.check_device_errors()


def test_command_lines_serve_the_design(tmp_path):
    """``random_model`` writes a folder from a config.json of the design; ``generate`` continues a prompt greedily as the
    plain implementation does and samples the same tokens for the same seed; ``bench_server`` runs its users."""
    import json
    import os
    import re
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

    def run_cli(module, *args):
        env = dict(os.environ, PYTHONPATH=root + os.pathsep + os.environ.get("PYTHONPATH", ""))
        proc = subprocess.run([sys.executable, "-m", module, *map(str, args)], stdout=subprocess.PIPE, stderr=subprocess.PIPE,
                              text=True, env=env, timeout=600, cwd=root)
        assert proc.returncode == 0, proc.stderr[-3000:]
        return proc.stdout

    cfg = config("A")
    cfg_path = str(tmp_path / "config.json")
    with open(cfg_path, "w") as f:
        json.dump(cfg, f)
    d = str(tmp_path / "model")
    run_cli("lightllm_b200.cli.random_model", cfg_path, d, 4, "--store-dtype", "float32")
    from tests.plain.qwen2_plain import read_safetensors
    w = {k: v.double() for k, v in read_safetensors(os.path.join(d, "model.safetensors")).items()}
    prompt = [5, 17, 3, 99, 250, 7]
    pick = lambda s: re.search(r"generated:\s*([\d ]+)", s).group(1)
    out = run_cli("lightllm_b200.cli.generate", d, *prompt, "--temperature", 0, "--max-new-tokens", 8, "--dtype", "float32",
                  "--max-seq-len", 64)
    got = [int(t) for t in pick(out).split()]
    assert len(got) == 8
    lg = P.forward(prompt + got, cfg, w)[0]
    for i, tok in enumerate(got):
        row = lg[len(prompt) - 1 + i]
        assert tok == int(torch.argmax(row)) or float(row.max() - row[tok]) < 1e-4, (got, i)
    a = run_cli("lightllm_b200.cli.generate", d, 1, 2, 3, "--seed", 5, "--max-seq-len", 64)
    b = run_cli("lightllm_b200.cli.generate", d, 1, 2, 3, "--seed", 5, "--max-seq-len", 64)
    assert pick(a) == pick(b)
    out = run_cli("lightllm_b200.cli.bench_server", d, 128, 64)
    assert "Hidden dim=44" in out and "vocab=303" in out
