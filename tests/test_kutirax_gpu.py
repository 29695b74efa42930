"""Kutirax on the GPU: every new kernel alone against the plain functions, then the model through the engine's own step
function, cache manager, scheduler and replay tool against the plain implementation, on five tiny configurations and on
configurations drawn at random."""
import random

import numpy as np
import pytest
import torch

from lightllm_b200 import Engine, EngineCore, EngineOptions, StepEntry
from lightllm_b200.csrc import ops
from tests.kutirax_configs import CONFIGS, PAGE_SIZE, config, random_config, random_weights, write_model
from tests.plain import kutirax_plain as P
from tests.tolerances import FLOAT32_ATOL, KUTIRAX_BF16_WORST_REL, logits_std, record
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


def single(parts):
    return all(b - a == 1 for _, _, a, b in parts)


# ---------------------------------------------------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D", [44, 50, 128, 896, 1537])
def test_norms_with_a_token_shift(dtype, D):
    """norm1, the shift towards the row before and norm2 in one launch: spans that begin a request, continue one, single
    tokens, a slot that a finished request used; the neighbouring floats of a slot stay as they are."""
    torch.manual_seed(D)
    x = {r: torch.randn(n, D) * 3 for r, n in (("a", 23), ("b", 12), ("c", 5))}
    w1, w2, mix = 1 + 0.2 * torch.randn(D), 1 + 0.2 * torch.randn(D), torch.randn(D)
    want1 = {r: P.token_shift(P.unit_rms(v.double(), 1e-5) * w1.double(), mix.double()) for r, v in x.items()}
    want2 = {r: P.unit_rms(v.double(), 1e-5) * w2.double() for r, v in x.items()}
    pre = 4 if D % 4 == 0 else 3
    state = torch.full((3, pre + D + (4 if D % 4 == 0 else 2)), NAN, device=DEV)

    def run(parts, second=True):
        rows = dev(torch.cat([x[r][a:b] for r, _, a, b in parts]))
        o1, o2 = torch.empty(rows.shape, dtype=DT[dtype], device=DEV), torch.empty(rows.shape, dtype=DT[dtype], device=DEV)
        clear = torch.full_like(rows, NAN) if second else None
        ops.norm_shift(rows, dev(w1), dev(mix), 1e-5, spans_of(parts), state, pre, o1, dev(w2) if second else None,
                       o2 if second else None, clear)
        at = 0
        for r, _, a, b in parts:
            close(o1[at:at + b - a], want1[r][a:b], dtype, f"shifted {r}[{a}:{b}]", rel=None if dtype == "float32" else 5e-3)
            if second:
                close(o2[at:at + b - a], want2[r][a:b], dtype, f"second norm {r}[{a}:{b}]", rel=None if dtype == "float32" else 5e-3)
            at += b - a
        if second:
            assert float(clear.abs().max()) == 0.0

    run([("a", 0, 0, 10), ("c", 1, 0, 5)])                     # c ends here; its slot 1 is used again by b
    run([("a", 0, 10, 11), ("b", 1, 0, 1)])
    run([("b", 1, 1, 2), ("a", 0, 11, 12)], second=False)
    run([("b", 1, 2, 4), ("a", 0, 12, 23)])
    run([("b", 1, 4, 12)])
    assert torch.isnan(state[:2, :pre]).all() and torch.isnan(state[:2, pre + D:]).all() and torch.isnan(state[2]).all()


def test_token_shift_without_its_own_norm_kernel():
    """The filter on a normed stream that something else made: the general path (a convolution of two taps)."""
    from lightllm_b200.engine.batch import Span, StepContext
    from lightllm_b200.parts.base import CacheView
    from lightllm_b200.parts.input_conv import TokenShift
    torch.manual_seed(0)
    D = 50
    part = TokenShift("l.shift", D, weight_name="")
    mix, h = torch.randn(D), torch.randn(9, D)
    part.bind({"l.shift": dev(mix)}, torch.float32, DEV)
    want = P.token_shift(h.double(), mix.double())
    state = torch.full((1, D + 2), NAN, device=DEV)
    for a, b in ((0, 4), (4, 5), (5, 9)):
        ctx = StepContext()
        ctx.device, ctx.spans, ctx.decode_only = DEV, [Span("a", 0, a, b - a, 0)], b - a == 1
        ctx.span_row, ctx.span_len, ctx.span_pos, ctx.span_slot, _ = spans_of([("a", 0, a, b)])
        close(part.forward(dev(h[a:b]), ctx, CacheView(None, None, None, state, True, 2), torch.float32), want[a:b], "float32", f"[{a}:{b}]")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,taps", [(13, 3), (64, 4), (40, 1), (36, 2), (260, 5), (12, 8)])
def test_convolution_with_bias_and_silu(dtype, C, taps):
    torch.manual_seed(C + taps)
    lens = {"a": 90, "b": 14, "c": 9}
    extra = 4
    proj = {r: torch.randn(n, C + 2 * extra).to(DT[dtype]) for r, n in lens.items()}
    w, b = torch.randn(C, taps), torch.randn(C)
    want = {r: P.silu(P.causal_conv(v.double()[:, extra:extra + C], w.double(), b.double())) for r, v in proj.items()}
    state = torch.full((3, 4 + (taps - 1) * C), NAN, device=DEV)

    def run(parts, fuse=False):
        rows = dev(torch.cat([proj[r][a:b] for r, _, a, b in parts]))
        out = torch.empty(rows.shape[0], C, dtype=DT[dtype], device=DEV)
        sp = spans_of(parts)
        ops.conv_act(rows, extra, C, dev(w), dev(b), "silu", sp, state if taps > 1 else None, 4, out, fuse_tail=fuse)
        if taps > 1 and not fuse:
            ops.conv_tail_update(rows, extra, C, taps, sp, state, 4)
        at = 0
        for r, _, p, q in parts:
            close(out[at:at + q - p], want[r][p:q], dtype, f"{r}[{p}:{q}]", rel=None if dtype == "float32" else 5e-3)
            at += q - p

    run([("a", 0, 0, 10), ("c", 1, 0, 9)])                       # c ends here; its slot 1 is used again by b
    run([("a", 0, 10, 11), ("b", 1, 0, 1)], fuse=True)
    run([("b", 1, 1, 2), ("a", 0, 11, 12)])
    run([("b", 1, 2, 3), ("a", 0, 12, 13)], fuse=True)
    run([("b", 1, 3, 5), ("a", 0, 13, 88)])
    run([("b", 1, 5, 14), ("a", 0, 88, 90)])
    if taps > 1:
        assert torch.equal(state[0, 4:].view(taps - 1, C).cpu(), proj["a"][90 - (taps - 1):, extra:extra + C].float())


# (heads, groups, state, vdim): every split of the walking kernel, the step kernel with and without whole pieces of four
# columns, the chunk kernels' three row heights and three column widths with sizes that do not fill them
SSM_SIZES = [(3, 1, 6, 10), (4, 2, 10, 6), (4, 2, 64, 32), (2, 1, 128, 64), (2, 1, 256, 72), (3, 3, 24, 16), (8, 4, 130, 4), (2, 2, 40, 8),
             (1, 1, 8, 8), (2, 1, 200, 24), (1, 1, 300, 12)]


@pytest.mark.parametrize("H,G,N,vd", SSM_SIZES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_space_over_spans_pieces_and_slots(dtype, H, G, N, vd):
    """The recurrence over three requests in several launches: one from its first token, one that continues from the state
    another launch left (in a slot that a finished request used), single tokens; long spans in one piece and in pieces that
    run side by side (bfloat16 inputs); the state lies behind other floats of its slot.  The inputs are what the kernels
    read, so the result is judged as float32 in both precisions."""
    inner, gn = H * vd, G * N
    C = inner + 2 * gn
    on_chunks = dtype == "bfloat16" and ops.state_space_chunks_support(N, vd, C, 0, inner, inner + gn)
    assert on_chunks == (dtype == "bfloat16" and N % 8 == 0 and vd % 8 == 0 and N <= 256)
    torch.manual_seed(H * N + vd)
    lens = {"a": 330, "b": 150, "c": 18}
    data = {r: ((torch.randn(n, C) * 0.5).to(DT[dtype]), torch.randn(n, H + 2).to(DT[dtype])) for r, n in lens.items()}
    data["a"][1][40:60] = 6.0                            # a stretch that forgets within a token or two
    bias, A, D = torch.randn(H) - 2.0, torch.randn(H) - 0.5, torch.randn(H)
    want = {}
    for r, (xbc, dt) in data.items():
        n, v = lens[r], xbc.double()
        d = torch.nn.functional.softplus(dt.double()[:, 1:1 + H] + bias.double(), threshold=200.0)
        want[r] = P.state_space(v[:, :inner].reshape(n, H, vd), v[:, inner:inner + gn].reshape(n, G, N),
                                v[:, inner + gn:].reshape(n, G, N), d, A.double(), D.double())
    for chunk in (None, 64, 128, 1 << 30) if on_chunks else (None,):
        run_state_space(data, want, bias, A, D, H, G, N, vd, chunk)


def run_state_space(data, want, bias, A, D, H, G, N, vd, chunk):
    off, size, inner, gn = 4, H * N * vd, H * vd, G * N
    state = torch.full((4, (off + size + 4) // 4 * 4 + 4), NAN, device=DEV)
    got = {}

    def run(parts):
        src = dev(torch.cat([data[r][0][a:b] for r, _, a, b in parts]))
        dt = dev(torch.cat([data[r][1][a:b] for r, _, a, b in parts]))
        out = torch.full((src.shape[0], inner), NAN, device=DEV)
        one = single(parts)
        ops.state_space(src, 0, inner, inner + gn, dt[:, 1:1 + H], dev(bias), dev(torch.exp(A)), dev(D), spans_of(parts), H, G, N, vd,
                        state, off, out, single=one, pieces=None if chunk is None or one else pieces_of(parts, chunk))
        at = 0
        for r, _, a, b in parts:
            got[(r, a, b)] = out[at:at + b - a].view(b - a, H, vd).cpu()
            at += b - a

    run([("a", 2, 0, 150), ("c", 0, 0, 18)])                   # c ends here; its slot 0 is used again by b
    run([("a", 2, 150, 151), ("b", 0, 0, 1)])
    run([("b", 0, 1, 3), ("a", 2, 151, 152)])
    run([("a", 2, 152, 153), ("b", 0, 3, 4)])
    run([("b", 0, 4, 150), ("a", 2, 153, 330)])
    for (r, a, b), o in got.items():
        scale = float(want[r].abs().max())
        err = float((o.double() - want[r][a:b]).abs().max())
        assert err <= 4e-5 * scale, f"state space {r}[{a}:{b}], pieces of {chunk}: {err:.3e} of {scale:.3e}"
    assert torch.isnan(state[2, :off]).all() and torch.isnan(state[2, off + size:]).all()
    assert torch.isfinite(state[2, off:off + size]).all() and torch.isnan(state[1]).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size,parts", [(10, 3), (30, 1), (64, 2), (4, 8), (1536, 2), (5000, 1)])
def test_gated_group_norm(dtype, size, parts):
    torch.manual_seed(size)
    T, n = 6, size * parts
    y, w = torch.randn(T, n) * 3, 1 + 0.2 * torch.randn(n)
    wide = torch.randn(T, n + 8).to(DT[dtype])
    want = P.gated_group_norm(y.double(), wide.double()[:, :n], w.double(), parts, 1e-5)
    out = torch.empty(T, n, device=DEV, dtype=DT[dtype])
    ops.gated_group_norm(dev(y), dev(wide)[:, :n], dev(w), parts, 1e-5, out)
    close(out, want, dtype, "gated norm", rel=None if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("qr,r,rd", [(18, 22, 6), (64, 96, 16), (8, 8, 8), (300, 512, 64)])
def test_latent_prepare(dtype, qr, r, rd):
    torch.manual_seed(qr)
    T = 9
    src = torch.randn(T, qr + r + rd + 3).to(DT[dtype])
    wq, wc = 1 + 0.2 * torch.randn(qr), 1 + 0.2 * torch.randn(r)
    pos = [3, 4, 5, 0, 1, 1000, 40001, 7, 8]
    freq = 500.0 ** (-torch.arange(0, rd, 2, dtype=torch.float64) / rd)
    slots = [4, 0, 1, 9, 3, 2, -1, 11, 6]
    cache = torch.full((12, 1, r + rd), NAN, device=DEV, dtype=DT[dtype])
    q = torch.empty(T, qr, device=DEV, dtype=DT[dtype])
    ops.latent_prepare(dev(src), 0, qr, qr + r, qr, r, rd, dev(wq), dev(wc), dev(freq.float()), False, i32(pos), i32(slots), q, cache, 1e-5)
    x = src.double()
    close(q, P.unit_rms(x[:, :qr], 1e-5) * wq.double(), dtype, "query latent", rel=None if dtype == "float32" else 5e-3)
    ang = torch.tensor(pos, dtype=torch.float64)[:, None] * freq
    u, v = x[:, qr + r:qr + r + rd // 2], x[:, qr + r + rd // 2:qr + r + rd]
    rot = torch.cat([u * ang.cos() - v * ang.sin(), v * ang.cos() + u * ang.sin()], -1)
    want = torch.cat([P.unit_rms(x[:, qr:qr + r], 1e-5) * wc.double(), rot], -1)
    for t, s in enumerate(slots):
        if s >= 0:          # (float32 angles at position 40,001 are good to about 2e-3 of a radian in the fastest pair)
            close(cache[s, 0], want[t], dtype, f"cache row of token {t}", rel=(4e-3 if pos[t] > 10000 else 1e-4) if dtype == "float32" else 1e-2)
    assert torch.isnan(cache[[5, 7, 8, 10]].float()).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,inn,on,rd", [(3, 3, 10, 22, 6), (40, 6, 32, 96, 16), (1, 2, 64, 256, 32), (130, 3, 64, 40, 8), (17, 5, 24, 512, 64),
                                          (70, 4, 96, 50, 0), (16, 2, 200, 8, 0)])
def test_per_head_contraction_with_a_rotated_part(dtype, T, H, inn, on, rd):
    torch.manual_seed(T + on)
    x = torch.randn(T, H * (inn + rd)).to(DT[dtype])
    w = (torch.randn(H, on, inn) / inn ** 0.5).to(DT[dtype])
    pos = torch.arange(5, 5 + T)
    out = torch.full((T, H * (on + rd)), NAN, device=DEV, dtype=DT[dtype])
    freq = 50.0 ** (-torch.arange(0, max(rd, 2), 2, dtype=torch.float64) / max(rd, 2))
    ops.head_linear(dev(x), 0, dev(w), out, x_head=inn + rd, out_head=on + rd,
                    rotate=(inn, on, rd, i32(pos.tolist()), dev(freq.float()), False) if rd else None)
    xh = x.double().view(T, H, inn + rd)
    got = out.view(T, H, on + rd)
    close(got[..., :on], torch.einsum("thi,hoi->tho", xh[..., :inn], w.double()), dtype, "contraction", rel=None if dtype == "float32" else 5e-3)
    if rd:
        ang = (pos.double()[:, None] * freq)[:, None]
        u, v = xh[..., inn:inn + rd // 2], xh[..., inn + rd // 2:]
        close(got[..., on:], torch.cat([u * ang.cos() - v * ang.sin(), v * ang.cos() + u * ang.sin()], -1), dtype, "rotation",
              rel=1e-4 if dtype == "float32" else 5e-3)


def latent_case(H, W, r, window, lens, starts, page, dtype, edge=None):
    """Requests with ``starts`` tokens in the cache bring ``lens`` rows of queries; pages that the window has passed are given
    back, rows no token has written hold NaN.  ``edge``: the last row's first head looks at one key with a score that stands
    out, ``edge`` positions before its own."""
    g = torch.Generator().manual_seed(H * W + sum(lens) + (edge or 0))
    S, T = len(lens), sum(lens)
    maxp = max(-(-(s + n) // page) for s, n in zip(starts, lens)) + 1
    pages = torch.randperm(S * maxp + 3, generator=g)[:S * maxp].view(S, maxp)
    cache = torch.full(((S * maxp + 3) * page, 1, W), NAN, dtype=DT[dtype])
    bt = torch.full((S, maxp), -1, dtype=torch.int32)
    q = torch.randn(T, H, W, generator=g).to(DT[dtype])
    scale, row, want = 1.5 * W ** -0.5, 0, []
    for i, (n, s) in enumerate(zip(lens, starts)):
        k = torch.randn(s + n, W, generator=g).to(DT[dtype])
        if edge is not None:
            target = s + n - 1 - edge
            if 0 <= target:
                q[row + n - 1, 0] = (k[target].float() * 6.0).to(DT[dtype])
        lo = max(0, s - window + 1) if window else 0
        for j in range(-(-(s + n) // page)):
            if (j + 1) * page > lo:
                bt[i, j] = pages[i, j]
                a, b = j * page, min(s + n, (j + 1) * page)
                cache[pages[i, j] * page:pages[i, j] * page + b - a, 0] = k[a:b]
        for t in range(n):
            pos = s + t
            first = max(0, pos - window + 1) if window else 0
            kk = k[first:pos + 1].double()
            p = torch.softmax((q[row + t].double() @ kk.T) * scale, -1)
            want.append(p @ kk[:, :r])
        row += n
    rows = np.cumsum([0] + list(lens))[:-1]
    args = (i32(rows), i32(lens), i32(starts), S, dev(bt), maxp, page)
    return dev(q).view(T, H * W), dev(cache), torch.stack(want), args, scale


def run_latent(kind, q, cache, args, H, W, r, window, scale, nsplit=1):
    T = q.shape[0]
    out = torch.full((T, H * r), NAN, device=DEV, dtype=q.dtype)
    one = T == args[3]
    if kind == "tcgen05":
        ops.latent_attention_tcgen05(q, cache, out, *args, H, W, r, window, scale)
    elif kind == "mma":
        ops.latent_attention(q, cache, out, *args, H, W, r, window, scale, one, nsplit)
    else:          # the CUDA-core kernel over value rows inside the key rows
        span_row, span_len, span_pos, S, bt, maxp, page = args
        lens = span_len.cpu().tolist()
        bq = 1 if one or nsplit > 1 else 2
        tiles = [(i, t) for i, n in enumerate(lens) for t in range(0, n, bq)]
        scratch = torch.empty(ops.attention_scratch_floats(len(tiles), H, r, bq, nsplit), device=DEV) if nsplit > 1 else None
        ops.paged_attention_simt(q, cache, cache, out, i32(t[0] for t in tiles), i32(t[1] for t in tiles), len(tiles), span_row, span_len,
                                 span_pos, bt, maxp, page, H, 1, W, window, scale, bq, nsplit, scratch, v_head_dim=r, v_stride=W)
    ops.check_async_errors(DEV)
    return out.view(T, H, r)


LATENT_SHAPES = [(6, 184, 144, 120, (40, 2, 300, 1), (0, 500, 77, 119), 16), (14, 288, 256, 100, (130, 5), (200, 0), 16),
                 (5, 72, 40, 0, (130, 5), (20, 3), 8), (3, 320, 256, 64, (65, 2), (1000, 63), 64), (40, 96, 64, 1000, (33,), (1500,), 32),
                 (1, 8, 8, 3, (70,), (5,), 16), (2, 24, 24, 17, (64, 64), (64, 63), 16), (17, 40, 8, 1, (9, 2), (0, 31), 8)]


@pytest.mark.parametrize("H,W,r,window,lens,starts,page", LATENT_SHAPES)
def test_latent_attention_of_portions(H, W, r, window, lens, starts, page):
    """Portions that begin and end inside pages and tiles, requests of unequal length in one launch, windows of one token up
    to more than the context, both tensor-core kernels and the CUDA-core one."""
    q, cache, want, args, scale = latent_case(H, W, r, window, lens, starts, page, "bfloat16")
    for kind in ("tcgen05", "mma", "simt"):
        close(run_latent(kind, q, cache, args, H, W, r, window, scale), want, "bfloat16", kind)
    q, cache, want, args, scale = latent_case(H, W, r, window, lens, starts, page, "float32")
    close(run_latent("simt", q, cache, args, H, W, r, window, scale), want, "float32", "simt")


@pytest.mark.parametrize("H,W,r,window,starts,page", [(6, 184, 144, 120, (500, 0, 119, 120), 16), (40, 576, 512, 0, (700, 90), 16),
                                                      (17, 40, 24, 50, (70,), 16), (70, 96, 64, 300, (63, 64, 1000), 8), (1, 16, 8, 1, (5, 0), 16)])
def test_latent_attention_of_single_tokens(H, W, r, window, starts, page):
    """Decoding: the keys whole and in pieces that a thread-block cluster merges (more pieces than tiles among them)."""
    lens = [1] * len(starts)
    q, cache, want, args, scale = latent_case(H, W, r, window, lens, starts, page, "bfloat16")
    for nsplit in (1, 2, 5, 8):
        close(run_latent("mma", q, cache, args, H, W, r, window, scale, nsplit), want, "bfloat16", f"{nsplit} pieces")
    close(run_latent("simt", q, cache, args, H, W, r, window, scale, 3), want, "bfloat16", "simt")


@pytest.mark.parametrize("window", [1, 16, 17, 63, 64, 65, 129, 200])
@pytest.mark.parametrize("last", [63, 64, 200, 333])
def test_a_key_just_inside_and_just_outside_the_window(window, last):
    """The last query matches one key with a score that stands out: at the window's edge it carries the row, one token further
    it must not be seen.  In a portion and as a single token, on every kernel."""
    H, W, r = 4, 72, 64
    for edge in (window - 1, window):
        if edge > last:
            continue
        for lens, starts in (((33,), (last - 32,)), ((1,), (last,))):
            q, cache, want, args, scale = latent_case(H, W, r, window, lens, starts, 16, "bfloat16", edge=edge)
            kinds = [("mma", 1), ("simt", 1)] + ([("tcgen05", 1)] if lens[0] > 1 else [("mma", 3)])
            for kind, nsplit in kinds:
                got = run_latent(kind, q, cache, args, H, W, r, window, scale, nsplit)
                close(got, want, "bfloat16", f"{kind}, key {edge} back under a window of {window}")
    # (the plain results on the two sides of the edge differ by far more than the tolerance)
    if window < last:
        inside = latent_case(H, W, r, window, (1,), (last,), 16, "bfloat16", edge=window - 1)[2]
        beside = latent_case(H, W, r, max(1, window - 1), (1,), (last,), 16, "bfloat16", edge=window - 1)[2]
        assert window == 1 or float((inside[0, 0] - beside[0, 0]).abs().max()) > 0.3


def test_latent_attention_sinks():
    H, W, r, window = 4, 72, 64, 50
    sinks = torch.tensor([0.0, 3.0, -2.0, 5.0])
    for lens, starts in (((20,), (90,)), ((1,), (100,))):
        q, cache, _, args, scale = latent_case(H, W, r, window, lens, starts, 16, "bfloat16")
        qq, T = q.view(-1, H, W).double().cpu(), q.shape[0]
        bt = args[4].cpu()[0]
        n = starts[0] + lens[0]
        want = torch.zeros(T, H, r, dtype=torch.float64)
        for t in range(T):
            pos = torch.arange(max(0, starts[0] + t - window + 1), starts[0] + t + 1)
            k = cache.cpu()[bt[pos // 16].long() * 16 + pos % 16, 0].double()
            s = torch.cat([(qq[t] @ k.T) * scale, sinks.double()[:, None]], -1)
            want[t] = torch.softmax(s, -1)[:, :-1] @ k[:, :r]
        for kind in ("mma", "tcgen05"):
            if kind == "tcgen05" and lens[0] == 1:
                continue
            out = torch.empty(T, H * r, device=DEV, dtype=torch.bfloat16)
            extra = (lens[0] == 1, 1) if kind == "mma" else ()
            fn = ops.latent_attention if kind == "mma" else ops.latent_attention_tcgen05
            fn(q, cache, out, *args, H, W, r, window, scale, *extra, sinks=dev(sinks))
            close(out.view(T, H, r), want, "bfloat16", kind)
        assert n > 0
    ops.check_async_errors(DEV)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,D,F", [(5, 44, 20), (40, 128, 192), (1, 50, 33), (300, 256, 512), (64, 64, 48), (129, 72, 1000)])
def test_squared_relu_feed_forward(dtype, T, D, F):
    from lightllm_b200.parts.mlp import PlainMLP
    torch.manual_seed(T + F)
    part = PlainMLP("m", D, F, names={"up": "up", "down": "down"}, weight_suffix="")
    W = {s.name: (torch.randn(s.shape) / s.shape[-1] ** 0.5).to(DT[dtype]) for s in part.weight_specs()}
    part.bind({k: dev(v) for k, v in W.items()}, DT[dtype], DEV)
    x = (torch.randn(T, D) * 2).to(DT[dtype])
    res = torch.zeros(T, D, device=DEV)
    part.forward(dev(x), res)
    close(res, P.squared_relu_mlp(x.double(), {k: v.double() for k, v in W.items()}, "m"), dtype, "feed-forward",
          rel=None if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("E,top", [(1, 1), (5, 2), (8, 8), (40, 3), (16, 1)])
def test_routing_by_the_softmax_over_the_chosen_logits(E, top):
    torch.manual_seed(E)
    T, D = 21, 44
    x, w, b = torch.randn(T, D), torch.randn(E, D), torch.randn(E) * 2
    ids, wts = P.route(x.double(), w.double(), b.double(), top)
    got_ids = torch.empty(T, top, dtype=torch.int32, device=DEV)
    got_w, dense = torch.empty(T, top, device=DEV), torch.empty(T, E, device=DEV)
    ops.moe_route(dev(x), dev(w), None, top, 1.0, got_ids, got_w, dense, softmax="chosen", bias=dev(b))
    assert torch.equal(got_ids.cpu().long(), ids)
    close(got_w, wts, "float32", "weights")
    full = torch.zeros(T, E, dtype=torch.float64).scatter(1, ids, wts)
    close(dense, full, "float32", "dense weights")
    # logits far apart: the weights of the chosen stay finite and sum to one
    ops.moe_route(dev(x * 300), dev(w), None, top, 1.0, got_ids, got_w, dense, softmax="chosen", bias=dev(b))
    assert torch.isfinite(got_w).all() and float((got_w.sum(-1) - 1).abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,D,E,top,ff", [(1, 64, 8, 2, 32), (3, 44, 5, 2, 12), (70, 64, 8, 2, 32), (40, 128, 4, 4, 16), (200, 64, 6, 3, 24)])
def test_routed_experts_part(dtype, T, D, E, top, ff):
    """Pair by pair, every expert on every row, grouped."""
    from lightllm_b200.parts.moe import RoutedExperts
    torch.manual_seed(T)
    part = RoutedExperts("m", D, ff, E, top, score="softmax_chosen", router_bias=True, bias_ending="b",
                         names={"gate": "gate", "up": "up", "down": "down", "router": "router"}, weight_suffix="", expert_prefix="e")
    W = {s.name: (torch.randn(s.shape) / s.shape[-1] ** 0.5).to(DT[dtype]) for s in part.weight_specs()}
    W["m.router.b"] = (2.0 * torch.randperm(E).float()).to(DT[dtype])
    W["m.router"] = (0.2 * W["m.router"].float()).to(DT[dtype])
    part.bind({k: dev(v) for k, v in W.items()}, DT[dtype], DEV)
    x = torch.randn(T, D).to(DT[dtype])
    res = torch.zeros(T, D, device=DEV)
    part.forward(dev(x), res)
    want = P.experts(x.double(), {"router": {"top": top}}, {k: v.double() for k, v in W.items()}, "m")
    close(res, want, dtype, "experts", rel=None if dtype == "float32" else 1.2e-2)


# ---------------------------------------------------------------------------------------------------------------------
# the model through the engine
# ---------------------------------------------------------------------------------------------------------------------
def make_model(tmp_path, name, dtype, seed=3, sharp=1.0, edit=None, cfg=None):
    cfg = config(name) if cfg is None else cfg
    for layer in cfg["layers"]:
        if layer["type"] == "latent_attention":
            layer["mixer"]["scale"] *= sharp
    w = random_weights(cfg, seed, store=DT[dtype], fixed_choice=dtype == "bfloat16")
    if edit is not None:
        edit(cfg, w)
    d = write_model(cfg, w, str(tmp_path / f"kut_{name}_{seed}_{dtype}"))
    return d, cfg, w


def core_for(d, dtype, name, pages=64, max_seqs=4, max_tokens=1024, graphs=True):
    return EngineCore(d, EngineOptions(dtype=dtype, max_seq_len=max_tokens, max_batch_tokens=max_tokens,
                                       page_size=PAGE_SIZE.get(name, 16), num_pages=pages, max_seqs=max_seqs, use_cuda_graphs=graphs))


def plain_logits(toks, w, cfg):
    return P.forward(cfg, w, toks).float()


def atol_for(name, dtype, plain):
    """float32: the largest difference of any logit, 1e-4 on logits of order one.  bfloat16: the root mean square over a
    row of logits (mean taken off), at most twice the worst that a recorded run showed, relative to the logits' spread."""
    std = logits_std(plain)
    return (FLOAT32_ATOL * max(1.0, std)) if dtype == "float32" else 2.0 * KUTIRAX_BF16_WORST_REL[name] * std


def error(got, plain, dtype) -> float:
    d = (got.double() - plain.double())
    if dtype == "float32":
        return float(d.abs().max())
    return float((d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt().max())


LENGTHS = {"A": [1, 2, 17, 33, 70, 150, 64, 49], "B": [3, 40, 131, 330, 129, 64, 257], "C": [1, 5, 40, 90, 33, 64, 17, 130],
           "D": [1, 3, 20, 45, 16, 70, 33, 9], "E": [2, 50, 140, 127, 64, 258]}


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
    worst = compare_with_plain(tr, got, plain, atol_for(name, dtype, once), f"Kutirax {name} {dtype}", rms=dtype != "float32")
    record(f"replay Kutirax {name} {dtype} ({len(tr.steps)} steps, pool for {tr.max_tokens} tokens)", worst, logits_std(once))


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
    """The attention alone decides: the recurrences' output projections, the feed-forwards' down projections and the shifts
    are zero."""
    for i, layer in enumerate(cfg["layers"]):
        for k in w:
            if k.startswith(f"l{i}.") and ((k.endswith("mix.o") and layer["type"] == "mamba2") or k.endswith(".down") or k.endswith(".shift")):
                w[k] = torch.zeros_like(w[k])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "D", "E"])
def test_sharp_attention_at_window_edges_and_page_borders(tmp_path, name, dtype):
    """The attention's scale multiplied by 4 and every other path into the stream silenced, so that single keys carry a row's
    output: the prompt in portions that end inside pages, then 60 tokens one by one, so that windows pass over decoded
    tokens.  The plain implementation itself, with every window one token longer or shorter, lies far outside the bound."""
    d, cfg, w = make_model(tmp_path, name, dtype, seed=8, sharp=4.0, edit=only_attention)
    rng = random.Random(2)
    n = {"B": 330, "E": 260}.get(name, 160)
    toks = [rng.randrange(cfg["vocab"]) for _ in range(n)]
    plain = plain_logits(toks, w, cfg)
    core = core_for(d, dtype, name)
    got = stepwise(core, "a", toks, [129, 2, 31, 2, 64] if name in "BE" else [9, 2, 16, 38, 2, 33])
    err = error(got, plain, dtype)
    record(f"sharp Kutirax {name} {dtype}", err, logits_std(plain))
    tol = atol_for(name + " sharp", dtype, plain)
    assert err <= tol
    core.runner.check_device_errors()
    for by in (-1, 1):
        off = {**cfg, "layers": [dict(l, mixer=dict(l["mixer"])) for l in cfg["layers"]]}
        for layer in off["layers"]:
            if layer["mixer"].get("mask"):
                layer["mixer"]["mask"] = {"size": layer["mixer"]["mask"]["size"] + by}
        assert error(plain_logits(toks, w, off), plain, dtype) > 1.5 * tol, by


def only_recurrence(cfg, w):
    """The recurrences alone decide, and they forget slowly; nothing is shifted."""
    for i, layer in enumerate(cfg["layers"]):
        for k in w:
            if not k.startswith(f"l{i}."):
                continue
            if (k.endswith("mix.o") and layer["type"] != "mamba2") or k.endswith(".down") or k.endswith(".shift"):
                w[k] = torch.zeros_like(w[k])
            if k.endswith("A_log"):
                w[k] = torch.full_like(w[k], -4.0)
            if k.endswith("dt_bias"):
                w[k] = torch.full_like(w[k], -1.0)


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
    record(f"recurrence Kutirax {name} {dtype}", err, logits_std(plain))
    tol = atol_for(name + " recurrence", dtype, plain)
    assert err <= tol
    off = error(plain_logits(toks[10:], w, cfg)[-20:], plain[-20:], dtype)
    assert off > 1.5 * tol, (off, tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_the_previous_token_is_carried_over_every_cut(tmp_path, name, dtype):
    """A shift of one (the mixer reads the token before, nothing of its own): a record of the previous input that is lost or
    stale at a portion's start moves the first logits after the cut; a plain run of the tokens behind the cut alone shows by
    how much."""
    def edit(cfg, w):
        for k in w:
            if k.endswith(".shift"):
                w[k] = torch.ones_like(w[k])
    d, cfg, w = make_model(tmp_path, name, dtype, seed=12, edit=edit)
    rng = random.Random(9)
    toks = [rng.randrange(cfg["vocab"]) for _ in range(60)]
    plain = plain_logits(toks, w, cfg)
    core = core_for(d, dtype, name)
    got = stepwise(core, "a", toks, [1, 2, 3, 16, 1, 1, 20])
    err = error(got, plain, dtype)
    record(f"shift Kutirax {name} {dtype}", err, logits_std(plain))
    tol = atol_for(name, dtype, plain)
    assert err <= tol
    assert error(plain_logits(toks[23:], w, cfg)[:1], plain[23:24], dtype) > 1.5 * tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_equals_token_by_token_and_long_decoding(tmp_path, name, dtype):
    """A whole prompt in one step against the same tokens one by one from the first (250 single steps: states, tails and the
    previous inputs are carried through every one, windows pass over decoded tokens, pages are given back and taken)."""
    d, cfg, w = make_model(tmp_path, name, dtype, seed=5)
    rng = random.Random(4)
    toks = [rng.randrange(cfg["vocab"]) for _ in range(250)]
    plain = plain_logits(toks, w, cfg)
    core = core_for(d, dtype, name)
    whole = stepwise(core, "a", toks, [250])
    one = stepwise(core, "b", toks, [])
    tol = atol_for(name, dtype, plain)
    record(f"Kutirax {name} {dtype} token by token", max(error(one, plain, dtype), error(whole, plain, dtype)), logits_std(plain))
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
        assert error(both, alone[r], dtype) <= (2e-5 * max(1.0, logits_std(plain)) if dtype == "float32" else tol), r
    record(f"Kutirax {name} {dtype} batch", worst, logits_std(plain))
    core.runner.check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tensor_core", [False, True])
def test_random_configurations_through_the_engine(tmp_path, dtype, tensor_core):
    for seed in range(5):
        cfg = random_config(random.Random(100 * seed + 7 * tensor_core), tensor_core)
        d, cfg, w = make_model(tmp_path, f"random{seed}", dtype, seed=seed, cfg=cfg)
        rng = random.Random(seed)
        toks = [rng.randrange(cfg["vocab"]) for _ in range(rng.choice([60, 120, 150]))]
        plain = plain_logits(toks, w, cfg)
        core = core_for(d, dtype, "random")
        got = stepwise(core, "a", toks, [rng.choice([2, 17, 33, 50]) for _ in range(3)])
        err = error(got, plain, dtype)
        record(f"random Kutirax {seed} {dtype} (tensor-core sizes: {tensor_core})", err, logits_std(plain))
        # (widths down to 24 leave few terms in every norm; a fault moves the logits by a large part of their spread)
        assert err <= (FLOAT32_ATOL * max(1.0, logits_std(plain)) if dtype == "float32" else 2.0 * KUTIRAX_BF16_WORST_REL["random"] * logits_std(plain)), (seed, cfg)
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
    margin_rel = 3e-4 if dtype == "float32" else 3.0 * KUTIRAX_BF16_WORST_REL[name]
    for p, o in zip(prompts, outs):
        lg = plain_logits(list(p) + o, w, cfg)
        for i, tok in enumerate(o):          # each token is the plain argmax given the same history
            row = lg[len(p) - 1 + i]
            top = torch.topk(row, 2).values
            assert tok == int(torch.argmax(row)) or float(top[0] - top[1]) < margin_rel * float(row.std()), (p, o, i)
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
    lg = P.forward(cfg, w, prompt + got)
    for i, tok in enumerate(got):
        top = torch.topk(lg[len(prompt) - 1 + i], 2).values
        assert tok == int(torch.argmax(lg[len(prompt) - 1 + i])) or float(top[0] - top[1]) < 1e-4, (got, i)
    a = run_cli("lightllm_b200.cli.generate", d, 1, 2, 3, "--seed", 5, "--max-seq-len", 64)
    b = run_cli("lightllm_b200.cli.generate", d, 1, 2, 3, "--seed", 5, "--max-seq-len", 64)
    assert pick(a) == pick(b)
    out = run_cli("lightllm_b200.cli.bench_server", d, 128, 64)
    assert "Hidden dim=44" in out and "vocab=301" in out
