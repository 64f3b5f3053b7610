"""The Nurasun family on the GPU against the plain implementation: each new kernel alone, each mechanism alone in a small
model, whole prompts against token-by-token decoding and portions down to two tokens, batches of unequal requests with
pages and slots used again, the first tokens of a sequence, the edges of chunks, keys far back, layers that read another
layer's cache, long decoding, greedy generation through the engine and its scheduler, the command line and the trace
replay.  Every test runs in 32-bit and in bfloat16."""

import copy
import os
import random
import subprocess
import sys

import pytest
import torch

import plain_nurasun as plain
from nurasun_models import MODELS, _lat, _model, make_nurasun_dir, steady_routers
import helpers
from helpers import BF16_NEAR_TIE, plain_inputs, random_tokens, run_trace
from test_gpu_fovunex import NEAR_TIE_NOISE, close, dev_i32, k, load, stepped
from test_gpu_gavatar import CLOSE_CALL, GavRef
from test_gpu_nurilorn import assert_close

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F = torch.float64


def reference(w, cfg, toks, dtype):
    """The plain model's logits, for bfloat16 how far rounding alone moves each row, and which rows rest on no close call
    of a router (a row whose own token is one is left out of a comparison)."""
    gaps = []
    logits = plain.forward(cfg, w, toks, gaps=gaps)
    keep = torch.ones(len(toks), dtype=torch.bool)
    if gaps:
        keep = torch.stack(gaps).min(dim=0).values >= CLOSE_CALL[dtype]
    if dtype == "float32":
        return GavRef(logits, None, keep)
    rounded = plain.forward(cfg, w, toks, round_to=torch.bfloat16)
    return GavRef(logits, (rounded - logits).norm(dim=-1) / logits.norm(dim=-1).clamp_min(1e-6), keep)


def routers_for(dtype):
    """In bfloat16 a router's input carries the rounding of everything before it; the whole-model runs in bfloat16 use
    routers that decide by a wide margin, the 32-bit runs keep the random ones (the route kernel is tested alone)."""
    return steady_routers if dtype == "bfloat16" else None


def steady_tokens(cfg, w, n: int, seed: int) -> list[int]:
    """``n`` random tokens on which the model is well conditioned: the plain model in 32-bit agrees with itself in 64-bit
    well within the bound that any implementation gets."""
    for s in range(seed, seed + 50):
        toks = random_tokens(cfg["vocab"], n, s)
        a, b = plain.forward(cfg, w, toks), plain.forward_float32(cfg, w, toks)
        if float((a - b).abs().max()) <= 0.25 * helpers.tolerance("float32", a):
            return toks
    raise AssertionError("no well-conditioned sequence in 50 seeds")


# =============================================================== kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, top", [(37, 1), (60, 3), (96, 2), (105, 4), (192, 1), (2048, 2), (1028, 1), (20480, 3)])
def test_sums_of_several_sublayers_with_the_dynamic_tanh_that_follows(dtype, d, top):
    """residual += mult * (y or a weighted sum of several y, plus up to two more rows) and tanh(alpha x) gain + offset of
    the new rows; the sum alone; the norm alone; gathered rows, which leave the residual as it was."""
    dt = TORCH[dtype]
    g = torch.Generator().manual_seed(d + top)
    n, mult, alpha = 6, 0.37, 0.8
    res = torch.randn(n, d, generator=g) * (0.2 + 3 * torch.rand(n, d, generator=g))
    gain, bias = torch.randn(d, generator=g).to(dt), torch.randn(d, generator=g).to(dt)
    weights = {"norm": gain, "norm.b": bias, "norm.alpha": torch.tensor(alpha)}
    tanh = (alpha, bias.to(DEV))
    pad = 0 if d % 4 == 0 and d > 100 else 3                # rows with and without a stride of their own
    for with_weights in ([False, True] if top == 1 else [True]):
        yt = torch.float32 if with_weights else dt
        y = torch.randn(n * top, d + pad, generator=g).to(yt)
        wts = torch.rand(n, top, generator=g) if with_weights else None
        add = y.double()[:, :d]
        if with_weights:
            add = (add.reshape(n, top, d) * wts.double()[:, :, None]).sum(1)
        for n_extra in (0, 1, 2):
            extras = [torch.randn(n, d + pad, generator=g).to(dt) for _ in range(n_extra)]
            total = add + sum((e.double()[:, :d] for e in extras), torch.zeros(n, d, dtype=F))
            want_res = res.double() + mult * total
            want = plain.tanh_norm(want_res, weights, "norm")
            args = (y.to(DEV)[:, :d], None, wts.to(DEV) if with_weights else None)
            more = dict(mult=mult, extras=tuple(e.to(DEV)[:, :d] for e in extras))
            rd, out = res.to(DEV), torch.empty(n, d, dtype=dt, device=DEV)
            k().stream_norm(rd, *args, gain.to(DEV), 1, 0.0, out, tanh=tanh, **more)
            assert torch.allclose(rd.double().cpu(), want_res, atol=1e-5, rtol=1e-5) and close(out, want, dtype, rel=1e-2)
            alone = res.to(DEV)
            k().stream_norm(alone, *args, None, 1, 0.0, None, **more)
            assert torch.equal(alone, rd)
            rows = [4, 0, 4, 5]
            rd2, some = res.to(DEV), torch.empty(4, d, dtype=dt, device=DEV)
            k().stream_norm(rd2, *args, gain.to(DEV), 1, 0.0, some, row_index=dev_i32(rows), tanh=tanh, **more)
            assert torch.equal(rd2.cpu(), res) and torch.equal(some, out[rows])
            # the same sum before a root mean square
            k().stream_norm(res.to(DEV), *args, gain.to(DEV), 1, 0.1, out, **more)
            assert close(out, plain.rms(want_res, gain, 0.1), dtype, rel=1e-2)
    rd, out = res.to(DEV), torch.empty(n, d, dtype=dt, device=DEV)
    k().stream_norm(rd, None, None, None, gain.to(DEV), 1, 0.0, out, tanh=tanh)
    assert torch.equal(rd.cpu(), res) and close(out, plain.tanh_norm(res.double(), weights, "norm"), dtype, rel=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("qh, kh, hd, rot, tied, biased", [
    (4, 2, 16, 16, True, True),          # sizes that the 16-byte form takes in bfloat16
    (6, 3, 64, 32, True, True),
    (3, 1, 40, 16, True, False),
    (2, 2, 24, 0, True, True),           # nothing turned
    (5, 1, 128, 128, False, True),       # no values of its own
    (5, 1, 9, 6, True, True),            # sizes that only the other form takes
    (4, 2, 16, 8, True, True),
    (3, 3, 12, 12, True, False),
    (40, 8, 64, 64, True, True),
])
@pytest.mark.parametrize("n", [7, 1100])
def test_biases_rotation_and_keys_that_are_the_values(dtype, qh, kh, hd, rot, tied, biased, n):
    """Biases, a rotation in halves at positions up to a million, keys and values (the keys before their rotation) into
    scattered slots; a padding token writes nothing; columns beside the heads stay."""
    dt = TORCH[dtype]
    if n > 100 and (qh > 10 or hd > 100):
        n = 600
    g = torch.Generator().manual_seed(hd + n)
    ps = 4
    pages = n // ps + 3
    pad = 8 if hd % 8 == 0 else 3
    q, kk = torch.randn(n, qh * hd + pad, generator=g).to(dt), torch.randn(n, kh * hd + pad, generator=g).to(dt)
    qb, kb = (torch.randn(h * hd, generator=g).to(dt) if biased else None for h in (qh, kh))
    positions = torch.randint(0, 3000, (n,), generator=g).tolist()
    positions[:4] = [0, 1, 1000003, 77]
    slots = torch.randperm(pages * ps, generator=g)[:n].tolist()
    slots[5] = -1
    mult = 1.3
    rd = {"base": 300.0, "dims": rot}

    def prep(x, heads, bias, turn):
        x = x.double()[:, :heads * hd] + (bias.double() if bias is not None else 0.0)
        x = x.reshape(n, heads, hd).clone()
        if rot and turn:
            for i in range(rot // 2):
                a = torch.tensor(positions, dtype=F)[:, None] * 300.0 ** (-2.0 * i / rot)
                u, v = x[:, :, i].clone(), x[:, :, i + rot // 2].clone()
                x[:, :, i], x[:, :, i + rot // 2] = (u * a.cos() - v * a.sin()) * mult, (v * a.cos() + u * a.sin()) * mult
        return x

    kpool = torch.full((pages, kh, ps, hd), 7.0, dtype=dt, device=DEV)
    vpool = torch.full((pages, kh, ps, hd), 7.0, dtype=dt, device=DEV)
    inv = (300.0 ** (-2.0 * torch.arange(rot // 2, dtype=F) / rot)).to(DEV) if rot else None
    qd, kd = q.to(DEV), kk.to(DEV)
    k().head_prepare(qd[:, :qh * hd], qh, hd, kd[:, :kh * hd], kh, hd, dev_i32(positions), dev_i32(slots), kpool, ps, inv_freq=inv,
                     rot_dims=rot, mult=mult, q_bias=qb.to(DEV) if biased else None, k_bias=kb.to(DEV) if biased else None,
                     tied=tied, vpool=vpool if tied else None)
    torch.cuda.synchronize()
    assert close(qd[:, :qh * hd].reshape(n, qh, hd), prep(q, qh, qb, True), dtype, rel=1e-2)
    assert torch.equal(qd[:, qh * hd:].cpu(), q[:, qh * hd:]) and torch.equal(kd.cpu(), kk)
    keep = torch.tensor([s >= 0 for s in slots])
    at = torch.tensor(slots)[keep]
    flat = lambda pool: pool.permute(0, 2, 1, 3).reshape(pages * ps, kh, hd).cpu()
    assert close(flat(kpool)[at], prep(kk, kh, kb, True)[keep], dtype, rel=1e-2)
    if tied:
        assert close(flat(vpool)[at], prep(kk, kh, kb, False)[keep], dtype, rel=1e-2)
    rest = torch.ones(pages * ps, dtype=torch.bool)
    rest[at] = False
    assert bool((flat(kpool)[rest] == 7.0).all()) and bool((flat(vpool)[rest if tied else slice(None)] == 7.0).all())


@pytest.mark.parametrize("M, N, K", [(1, 48, 72), (8, 96, 256), (16, 512, 512), (5, 1100, 1024), (200, 320, 128), (384, 512, 256), (129, 96, 64)])
def test_activations_in_the_epilogues_of_the_products(M, N, K):
    """The tanh form of gelu over alternating gate and up rows, and the square of relu, in the weight-streaming products
    (both kernels) and in the tcgen05 product; gates from far below to far above zero."""
    g = torch.Generator().manual_seed(M + N)
    bf = torch.bfloat16
    a = torch.randn(M, K, generator=g).to(bf)
    w = (torch.randn(N, K, generator=g) * (2.0 / K ** 0.5)).to(bf)
    w[0] *= 40                                                  # a gate whose third power leaves float32's exponent range
    ref = a.double() @ w.double().T
    half, full = torch.full((M, N // 2), float("nan"), device=DEV, dtype=bf), torch.full((M, N), float("nan"), device=DEV, dtype=bf)
    act = k().glu_constants("gelu_tanh")
    if M <= 16:
        k().gemm_stream(a.to(DEV), w.to(DEV), half, M, "glu", act=act)
        k().gemm_stream(a.to(DEV), w.to(DEV), full, M, "relu2")
        assert k().stream_error() == 0
    else:
        k().gemm_tcgen05(a.to(DEV), w.to(DEV), half, "silu_mul", act=act)
        k().gemm_tcgen05(a.to(DEV), w.to(DEV), full, "relu2")
        torch.cuda.synchronize()
        assert k().gemm_tcgen05_error() == 0
    want = plain.gelu(ref[:, 0::2]) * ref[:, 1::2]
    assert float((ref[:, 0] < -8).double().mean()) > 0 or M == 1
    for got, want in ((half, want), (full, torch.relu(ref) ** 2)):
        scale = want.abs().amax(dim=0).clamp_min(1.0)           # column by column: the first one is far larger than the others
        assert bool((((got.double().cpu() - want).abs() / scale).amax() <= 1e-2)), (M, N, K)


@pytest.mark.parametrize("dtype", DTYPES)
def test_activation_kernels_and_the_cap(dtype):
    dt = TORCH[dtype]
    g = torch.Generator().manual_seed(2)
    for n, d in ((5, 37), (3, 64), (33, 40)):
        gu = (3 * torch.randn(n, 2 * d, generator=g)).to(dt)
        gu[0, 0], gu[0, 1] = -60.0, 60.0
        for inter in (False, True):
            gate, up = (gu[:, 0::2], gu[:, 1::2]) if inter else (gu[:, :d], gu[:, d:])
            out = torch.empty(n, d, dtype=dt, device=DEV)
            k().glu_act(gu.to(DEV), out, "gelu_tanh", interleaved=inter)
            assert torch.isfinite(out).all() and close(out, plain.gelu(gate.double()) * up.double(), dtype, rel=1e-2)
        wide = (2 * torch.randn(n, d + 5, generator=g)).to(dt)
        out = torch.empty(n, d, dtype=dt, device=DEV)
        k().relu2(wide.to(DEV)[:, 2:2 + d], out)
        assert close(out, torch.relu(wide.double()[:, 2:2 + d]) ** 2, dtype, rel=1e-2)
        k().relu2(out, out)
        assert close(out, torch.relu(wide.double()[:, 2:2 + d]) ** 4, dtype, rel=2e-2)
        x = 20 * torch.randn(n, d, generator=g)
        xd = x.to(DEV)
        k().softcap(xd, 7.5)
        assert torch.allclose(xd.double().cpu(), 7.5 * torch.tanh(x.double() / 7.5), atol=1e-5, rtol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, ff, experts, top, shared", [(40, 24, 5, 2, 16), (72, 20, 3, 1, 0), (64, 136, 4, 3, 136), (64, 32, 6, 6, 200),
                                                         (48, 40, 1, 1, 24), (64, 128, 4, 3, 64), (192, 64, 7, 2, 128)])
@pytest.mark.parametrize("n", [1, 9, 20, 150])
def test_experts_without_a_gate_and_a_shared_one(dtype, d, ff, experts, top, shared, n):
    """Router, both grouped products on both of their kernels, the shared expert (a few rows and many), summed up by the
    part itself and left to the block."""
    from inf_engine_b200.config import MLPSpec, RoutedExpertsSpec
    from inf_engine_b200.parts import RoutedExperts, Runtime

    dt = TORCH[dtype]
    g = torch.Generator().manual_seed(d + n)
    rand = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).to(dt)
    w = {"router": 2 * rand(experts, d)}
    for e in range(experts):
        w[f"e{e}.up"], w[f"e{e}.down"] = 1.5 * rand(ff, d), rand(d, ff)
    if shared:
        w["shared.up"], w["shared.down"] = 1.5 * rand(shared, d), rand(d, shared)
    spec = RoutedExpertsSpec(kind="routed_experts", hidden=d, intermediate=ff, n_experts=experts, top=top, router="router",
                             expert_prefix="e", gated=False, activation="relu2",
                             shared=MLPSpec(kind="mlp", hidden=d, intermediate=shared, up_proj="shared.up", down_proj="shared.down") if shared else None)
    assert set(RoutedExperts.expected_tensors(spec)) == set(w)
    part = RoutedExperts(spec, {name: t.to(DEV) for name, t in w.items()}, Runtime(DEV, dt))
    x = torch.randn(n, d, generator=g).to(dt)
    mlp = {"router": {"experts": experts, "top": top}, "shared": {"ff": shared} if shared else None}
    gaps = []
    want = plain.mixture(x.double(), mlp, w, "", gaps=gaps)
    keep = gaps[0] > 1e-3
    out = part.forward(x.to(DEV), None).double().cpu()
    assert close(out[keep], want[keep], dtype, rel=1e-2)
    y, weights, more = part.forward_unsummed(x.to(DEV), None)
    total = (y.double().reshape(n, top, d) * weights.double()[:, :, None]).sum(1) + sum(m.double() for m in more)
    assert len(more) == bool(shared) and torch.allclose(total.cpu(), out, atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("n, d, ff, experts, top", [(300, 128, 192, 5, 2), (700, 64, 64, 9, 3), (129, 320, 64, 3, 1), (260, 64, 320, 2, 2)])
@pytest.mark.parametrize("bn", [128, 256])
def test_grouped_product_on_tcgen05(n, d, ff, experts, top, bn):
    """Experts with no row, with one, with exactly a tile's 128 and with several tiles; output widths that are no multiple
    of a tile's; rows gathered into sorted order, results in sorted order and in the pairs' own places; every epilogue."""
    bf = torch.bfloat16
    g = torch.Generator().manual_seed(n + ff)
    x = torch.randn(n, d, generator=g).to(bf)
    first, both, down = ((torch.randn(experts, *s, generator=g) / s[-1] ** 0.5).to(bf) for s in ((ff, d), (2 * ff, d), (d, ff)))
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(n)]).to(torch.int32)
    if top == 1:
        ids[:] = 2                                       # all in one expert, then one row and none in the others
        ids[5] = 0
    elif experts == 9:
        ids[:, 0] = 8                                    # 700 rows of one expert; the others' counts follow from the rest
        ids[:, 1] = torch.where(torch.arange(n) < 128, 1, 2)
        ids[:, 2] = torch.where(torch.arange(n) < 1, 3, 4)
    rows = k().gemm_tcgen05_tile_rows()
    P = n * top
    pairs = torch.empty(P, dtype=torch.int32, device=DEV)
    tiles = torch.full((k().moe_max_tiles(P, experts, rows), 4), -5, dtype=torch.int32, device=DEV)
    k().moe_sort(ids.to(DEV), experts, pairs, tiles, rows)
    counts = torch.bincount(ids.flatten().long(), minlength=experts)
    t, order = tiles.cpu(), pairs.cpu().long()
    assert int(t[0, 3]) == int((t[:, 2] > 0).sum()) == int((-(-counts // rows)).sum()) and int(t[:, 2].sum()) == P
    xs = torch.empty(P, d, dtype=bf, device=DEV)
    k().moe_gather(x.to(DEV), xs, pairs, top)
    assert torch.equal(xs.cpu(), x[order // top])
    expert_of = ids.flatten().long()[order]
    z = torch.einsum("pd,pfd->pf", xs.double().cpu(), first.double()[expert_of])
    zb = torch.einsum("pd,pfd->pf", xs.double().cpu(), both.double()[expert_of])
    h = torch.full((P, ff), float("nan"), dtype=bf, device=DEV)
    k().gemm_tcgen05_grouped(xs, first.to(DEV), h, tiles, None, "relu2", bn=bn)
    assert close(h, torch.relu(z) ** 2, "bfloat16", rel=1e-2)
    for act in (None, k().glu_constants("gelu_tanh"), (1.702, 0.9, 1.0)):
        k().gemm_tcgen05_grouped(xs, both.to(DEV), h, tiles, None, "silu_mul", act=act, bn=bn)
        gate, up = zb[:, 0::2], zb[:, 1::2]
        want = torch.nn.functional.silu(gate) * up if act is None else plain.gelu(gate) * up
        if act is not None and len(act) == 3:
            gate, up = gate.clamp(max=0.9), up.clamp(-0.9, 0.9)
            want = gate * torch.sigmoid(1.702 * gate) * (up + 1)
        assert close(h, want, "bfloat16", rel=1e-2), act
    y = torch.full((P, d), float("nan"), device=DEV)
    k().gemm_tcgen05_grouped(h, down.to(DEV), y, tiles, pairs, "f32", bn=bn)
    torch.cuda.synchronize()
    assert k().gemm_tcgen05_error() == 0
    want = torch.empty(P, d, dtype=F)
    want[order] = torch.einsum("pf,pdf->pd", h.double().cpu(), down.double()[expert_of])
    assert torch.isfinite(y).all() and close(y, want, "bfloat16", rel=2e-3)
    # the last rows of a wider result, and a result with a stride of its own
    wide = torch.full((P, d + 8), 3.0, device=DEV)
    k().gemm_tcgen05_grouped(h, down.to(DEV), wide[:, 4:4 + d], tiles, pairs, "f32", bn=bn)
    assert torch.equal(wide[:, 4:4 + d], y) and bool((wide[:, :4] == 3.0).all()) and bool((wide[:, 4 + d:] == 3.0).all())


@pytest.mark.parametrize("d, ff, experts, top, n", [(256, 64, 6, 2, 7), (72, 40, 4, 3, 16), (1024, 24, 3, 1, 1), (64, 520, 5, 5, 16)])
def test_experts_products_that_stream_their_weights(d, ff, experts, top, n):
    """The form for a few tokens beside the tiles' form, pair by pair, and against the plain products."""
    bf = torch.bfloat16
    g = torch.Generator().manual_seed(d + ff)
    x = torch.randn(n, d, generator=g).to(bf)
    first, down = ((torch.randn(experts, *s, generator=g) / s[-1] ** 0.5).to(bf) for s in ((2 * ff, d), (d, ff)))
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(n)]).to(torch.int32)
    pairs = torch.empty(n * top, dtype=torch.int32, device=DEV)
    tiles = torch.empty(k().moe_max_tiles(n * top, experts), 4, dtype=torch.int32, device=DEV)
    k().moe_sort(ids.to(DEV), experts, pairs, tiles)
    order = pairs.cpu().long()
    expert_of = ids.flatten().long()[order]
    outs = []
    for few in (True, False):
        # the number of rows of the result decides: a result with rows to spare takes the other form
        rows = n * top if few else (k().MOE_FEW_TOKENS + 1) * top
        h, h2 = torch.zeros(rows, ff, dtype=bf, device=DEV), torch.zeros(rows, 2 * ff, dtype=bf, device=DEV)
        y = torch.zeros(rows, d, device=DEV)
        k().moe_gemm(x.to(DEV), first.to(DEV), h, pairs, tiles, top, gather=True, scatter=False, epi="silu_mul")
        k().moe_gemm(x.to(DEV), first.to(DEV), h2, pairs, tiles, top, gather=True, scatter=False, epi="relu2")
        k().moe_gemm(h, down.to(DEV), y, pairs, tiles, top, gather=False, scatter=True)
        outs.append([t[:n * top].double().cpu() for t in (h, h2, y)])
    z = torch.einsum("pd,pfd->pf", x.double()[order // top], first.double()[expert_of])
    for h, h2, y in outs:
        assert close(h, torch.nn.functional.silu(z[:, 0::2]) * z[:, 1::2], "bfloat16", rel=1e-2)
        assert close(h2, torch.relu(z) ** 2, "bfloat16", rel=1e-2)
        want = torch.empty(n * top, d, dtype=F)
        want[order] = torch.einsum("pf,pdf->pd", h, down.double()[expert_of])
        assert close(y, want, "bfloat16", rel=2e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m, heads, kd, nd", [(1, 3, 10, 6), (8, 4, 192, 64), (16, 2, 64, 192), (9, 5, 17, 70), (3, 1, 300, 130), (12, 2, 40, 8)])
def test_per_head_products_of_a_few_rows(dtype, m, heads, kd, nd):
    dt = TORCH[dtype]
    g = torch.Generator().manual_seed(kd)
    x = torch.randn(m, heads * kd + 5, generator=g).to(dt)
    w = (torch.randn(heads, kd, nd, generator=g) / kd ** 0.5).to(dt)
    out = torch.full((m, heads * nd + 2), 7.0, dtype=dt, device=DEV)
    k().heads_gemm(x.to(DEV)[:, :heads * kd], kd, w.to(DEV), out[:, :heads * nd], nd)
    want = torch.einsum("mhk,hkn->mhn", x.double()[:, :heads * kd].reshape(m, heads, kd), w.double()).reshape(m, -1)
    assert close(out[:, :heads * nd], want, dtype, rel=1e-2) and bool((out[:, heads * nd:] == 7.0).all())
    alone = torch.empty(1, heads * nd, dtype=dt, device=DEV)      # a row's sum does not depend on the other rows
    k().heads_gemm(x.to(DEV)[m - 1:, :heads * kd], kd, w.to(DEV), alone, nd)
    assert torch.equal(alone[0], out[m - 1, :heads * nd])


def test_router_of_sigmoid_scores_without_groups():
    """Weights over their sum, ties to the lower index, scores that underflow."""
    for n_experts, top in ((6, 3), (40, 6), (5, 5), (1, 1)):
        g = torch.Generator().manual_seed(n_experts)
        z = 2 * torch.randn(33, n_experts, generator=g)
        z[0] = 1.0
        z[1] = torch.arange(n_experts) % 2
        z[2] = -200.0                                            # every score 0: the sum is the small constant
        z[3] = -60.0 - torch.arange(n_experts)
        ids = torch.empty(33, top, dtype=torch.int32, device=DEV)
        wts = torch.empty(33, top, dtype=torch.float32, device=DEV)
        k().moe_route(z.to(DEV), None, ids, wts, None, n_experts, top, 1, 1, 1.0, 1e-20, score="sigmoid")
        want, ww = plain.route(z.double(), {"experts": n_experts, "top": top}, {"router": torch.eye(n_experts, dtype=F)}, "")
        for t in range(33):
            if t == 2:
                assert float(wts[t].abs().max()) <= 1e-6
                continue
            assert ids[t].tolist() == want[t], (n_experts, t)
            assert torch.allclose(wts[t].double().cpu(), torch.tensor(ww[t], dtype=F), atol=1e-6, rtol=1e-5)


# =============================================================== whole models
LENGTH = {"sun_a": 97, "sun_b": 70, "sun_c": 131, "sun_w": 190, "sun_t": 280, "sun_att": 75, "sun_lat": 90, "sun_moe": 41, "sun_dense": 60}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_whole_prompt_decoding_and_portions_agree_with_the_plain_model(tmp_path, name, dtype):
    folder = make_nurasun_dir(tmp_path, name, fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    toks = steady_tokens(cfg, w, LENGTH[name], 21)
    ref = reference(w, cfg, toks, dtype)
    r = load(folder, dtype, page_size=8)
    T = len(toks)
    assert_close(stepped(r, "whole", toks, [T]), ref, dtype, f"{name}: whole")
    assert_close(stepped(r, "decode", toks, [T - 40] + [1] * 40), ref, dtype, f"{name}: decoded one by one")
    assert_close(stepped(r, "one", toks[:30], [1]), ref[:30], dtype, f"{name}: token by token from the start")
    assert_close(stepped(r, "cut", toks, [7, 2, 16, 3, 2, 17, 2, 31, 1, 5]), ref, dtype, f"{name}: portions")
    assert_close(stepped(r, "pairs", toks[:40], [2]), ref[:40], dtype, f"{name}: portions of two")
    r.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["sun_a", "sun_b"])
def test_stream_after_every_layer(tmp_path, name, dtype):
    """The residual stream layer by layer, not the logits alone: the model is cut after 1, 2, .. layers."""
    folder = make_nurasun_dir(tmp_path, name, fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    toks = steady_tokens(cfg, w, 33, 5)
    for n in range(1, len(cfg["layers"]) + 1):
        c = copy.deepcopy(MODELS[name])
        c["layers"] = c["layers"][:n]

        def fix(t):
            for tensor in list(t):
                t[tensor] = w[tensor].to(t[tensor].dtype)
        d = tmp_path / f"cut{n}"
        d.mkdir()
        part = make_nurasun_dir(d, name, config=c, fix=fix)
        cc, ww = plain_inputs(part)
        r = load(part, dtype, page_size=8)
        assert_close(stepped(r, "x", toks, [33]), reference(ww, cc, toks, dtype), dtype, f"{name}: after {n} layers")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["sun_a", "sun_b", "sun_c", "sun_w", "sun_t"])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(tmp_path, name, dtype):
    """Seven requests, at most three live, portions of some beside decoded tokens of others, some left out of a step;
    the pool holds exactly what the fullest moment needs and free pages are filled with NaN."""
    from inf_engine_b200 import StepEntry

    folder = make_nurasun_dir(tmp_path, name, fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    lengths = [45, 17, 80, 3, 33, 64, 1]
    reqs = {f"q{i}": steady_tokens(cfg, w, n, 40 + 100 * i) for i, n in enumerate(lengths)}
    refs = {rid: reference(w, cfg, t, dtype) for rid, t in reqs.items()}
    rng = random.Random(7)
    plan, waiting, live = [], list(reqs), {}
    while waiting or live:
        while waiting and len(live) < 3:
            rid = waiting.pop(0)
            live[rid] = [0, max(1, len(reqs[rid]) - rng.choice([2, 6, 12]))]
        step, ended = [], []
        for rid, st in list(live.items()):
            if rng.random() < 0.25 and len(live) > 1:
                continue
            n = 1 if st[0] >= st[1] else min(rng.choice([2, 3, 5, 11, 24]), st[1] - st[0])
            step.append((rid, st[0], n))
            st[0] += n
            if st[0] == len(reqs[rid]):
                ended.append(rid)
                del live[rid]
        if step:
            plan.append((step, ended))
    ps = 8
    held, most = {}, 0
    for step, ended in plan:
        for rid, p, n in step:
            held[rid] = -(-(p + n) // ps)
        most = max(most, sum(held.values()))
        for rid in ended:
            held.pop(rid)
    r = load(folder, dtype, page_size=ps, n_pages=max(most, 1), max_requests=3, poison_free_pages=True)
    got = {rid: [] for rid in reqs}
    slots_seen = {}
    for step, ended in plan:
        for rid, p, n in step:
            if not r.is_open(rid):
                assert r.open(rid)
                slots_seen[rid] = r.cache.slots[rid]
        lg = r.step([StepEntry(rid, reqs[rid][p:p + n], list(range(n))) for rid, p, n in step]).cpu()
        at = 0
        for rid, p, n in step:
            got[rid].append(lg[at:at + n].clone())
            at += n
        for rid in ended:
            r.close(rid)
        r.cache.check()
    assert len(set(slots_seen.values())) <= 3 < len(slots_seen)              # slots were used again
    for rid in reqs:
        assert_close(torch.cat(got[rid]), refs[rid], dtype, f"{name}: {rid} in mixed batches")


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_of_a_sequence_and_pages_that_another_request_held(tmp_path, dtype):
    """Sequences of one, two and three tokens in one batch; then new requests in the places they held."""
    from inf_engine_b200 import StepEntry

    folder = make_nurasun_dir(tmp_path, "sun_a", fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    r = load(folder, dtype, max_requests=3, n_pages=3, poison_free_pages=True)
    first = {"a": steady_tokens(cfg, w, 1, 1), "b": steady_tokens(cfg, w, 2, 100), "c": steady_tokens(cfg, w, 3, 200)}
    second = {"d": steady_tokens(cfg, w, 9, 300), "e": steady_tokens(cfg, w, 1, 400), "f": steady_tokens(cfg, w, 2, 500)}
    for batch in (first, second):
        for rid in batch:
            assert r.open(rid)
        lg = r.step([StepEntry(rid, t, list(range(len(t)))) for rid, t in batch.items()]).cpu()
        at = 0
        for rid, t in batch.items():
            assert_close(lg[at:at + len(t)], reference(w, cfg, t, dtype), dtype, f"first tokens of {rid}")
            at += len(t)
        for i, tok in enumerate([9, 9, 120]):
            rid, t = list(batch.items())[1]
            lg = r.step([StepEntry(rid, [tok], [0])]).cpu()
            assert_close(lg, reference(w, cfg, t + [9, 9, 120][:i + 1], dtype)[-1:], dtype, "second and later tokens")
        for rid in batch:
            r.close(rid)
        r.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["sun_att", "sun_a", "sun_b", "sun_c", "sun_w", "sun_t"])
def test_edges_of_the_chunks_in_prompts_and_in_decoding(tmp_path, name, dtype):
    """The attention is made sharp so that one key more or less changes the logits far beyond rounding; the sequence runs
    over several chunks, in pages of 8, so that pages behind a chunk are given back (and filled with NaN)."""
    config = copy.deepcopy(MODELS[name])
    for L in config["layers"]:
        if L["type"] == "attention":
            L["mixer"]["scale"] *= 2.5
    folder = make_nurasun_dir(tmp_path, name, config=config, fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    size = min(L["mixer"]["mask"]["size"] for L in cfg["layers"] if "mask" in L["mixer"])
    toks = steady_tokens(cfg, w, 3 * size + 5 if size > 10 else 41, 8)
    ref = reference(w, cfg, toks, dtype)
    # the faults this must catch: a chunk one position longer or shorter
    for delta in (1, -1):
        other = copy.deepcopy(cfg)
        for L in other["layers"]:
            if "mask" in L["mixer"]:
                L["mixer"]["mask"]["size"] += delta
        wrong = plain.forward(other, w, toks)
        moved = (wrong - ref.logits).norm(dim=-1).div(ref.logits.norm(dim=-1))[size - 1:]
        assert float(moved.max()) > 0.02, (delta, float(moved.max()))
    r = load(folder, dtype, page_size=8, poison_free_pages=True)
    noise = 1.5
    assert_close(stepped(r, "whole", toks, [len(toks)]), ref, dtype, f"{name}: chunk edges in a prompt", noise=noise)
    assert_close(stepped(r, "decode", toks, [3] + [1] * (len(toks) - 3)), ref, dtype, f"{name}: chunk edges in decoding", noise=noise)
    assert_close(stepped(r, "cut", toks, [size - 1, 2, 1, 1, 5, 11]), ref, dtype, f"{name}: portions around a chunk's edge", noise=noise)
    assert_close(stepped(r, "cut2", toks, [size, size + 1, 2]), ref, dtype, f"{name}: portions that end on an edge", noise=noise)
    r.cache.check()
    for g in r.cache.kv_groups:
        assert g.pool.n_free == g.pool.n_pages


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_token_is_seen_to_the_end_of_its_chunk_and_no_further(tmp_path, dtype):
    """One layer of attention: changing the token just inside a chunk's end, or the first of the next, moves the rows of
    its own chunk from its place on and leaves every other row as it was, bit for bit, however the prompt is cut."""
    folder = make_nurasun_dir(tmp_path, "sun_att")
    cfg, w = plain_inputs(folder)
    size, T = cfg["layers"][0]["mixer"]["mask"]["size"], 75
    toks = random_tokens(cfg["vocab"], T, 31)
    r = load(folder, dtype, page_size=8)
    for sizes in ([T], [1], [2], [size - 3, 5, 17, 2]):
        base = stepped(r, "base", toks, sizes)
        for at in (size - 1, size, 2 * size - 1):
            other = list(toks)
            other[at] = (toks[at] + 50) % cfg["vocab"]
            rows = (stepped(r, "other", other, sizes) - base).abs().amax(dim=-1)
            end = (at // size + 1) * size
            assert bool((rows[at:end] > 1e-4).all()), (sizes, at)
            rows[at:end] = 0
            assert float(rows.max()) == 0.0, (sizes, at)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["sun_lat", "sun_w", "sun_t"])
def test_a_far_key_is_found(tmp_path, name, dtype):
    """The attention is made sharp; the test first shows that swapping one token 250 and more positions back moves the
    last positions' plain logits, then the engine must agree with the plain model there, in a prompt, decoded and in
    portions (the kernels alone are tested with a key that dominates)."""
    config = copy.deepcopy(MODELS[name])
    for L in config["layers"]:
        if "mask" not in L["mixer"]:
            L["mixer"]["scale"] *= 3.0
    folder = make_nurasun_dir(tmp_path, name, config=config, fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    toks = steady_tokens(cfg, w, 300, 12)
    ref = reference(w, cfg, toks, dtype)
    swapped = list(toks)
    swapped[5] = (toks[5] + 17) % cfg["vocab"]
    moved = (plain.forward(cfg, w, swapped)[250:] - ref.logits[250:]).norm(dim=-1) / ref.logits[250:].norm(dim=-1)
    assert float(moved.max()) > 1e-3
    r = load(folder, dtype, page_size=8, n_pages=80)
    assert_close(stepped(r, "whole", toks, [300]), ref, dtype, "far key in a prompt", noise=1.5)
    assert_close(stepped(r, "decode", toks, [250] + [1] * 50), ref, dtype, "far key in decoding", noise=1.5)
    assert_close(stepped(r, "cut", toks, [64, 65, 2, 127, 3, 39]), ref, dtype, "far key in portions", noise=1.5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_readers_of_another_layers_vectors(tmp_path, dtype):
    """Two layers compress, two readers each, interleaved: a reader of the wrong one, or one that took this step's tokens
    only, shows (the readers' own sharp scores make up most of what is added)."""
    config = _model(97, 64, 1e-5, 1.0, None, [_lat(2, 16, 8, 32, 0.5, None), _lat(3, 8, 16, 32, 0.4, None),
                                              _lat(4, 16, 16, 32, 1.5, None, 1), _lat(1, 32, 40, 32, 1.0, None, 0),
                                              _lat(2, 12, 20, 32, 1.5, None, 0), _lat(5, 8, 8, 32, 1.5, None, 1)])
    folder = make_nurasun_dir(tmp_path, "readers", config=config)
    cfg, w = plain_inputs(folder)
    toks = steady_tokens(cfg, w, 70, 3)
    ref = reference(w, cfg, toks, dtype)
    for i, j in ((2, 0), (3, 1), (4, 1), (5, 0)):
        other = copy.deepcopy(cfg)
        other["layers"][i]["mixer"]["kv_from"] = j
        moved = (plain.forward(other, w, toks) - ref.logits).norm(dim=-1) / ref.logits.norm(dim=-1)
        assert float(moved.max()) > 0.05, (i, float(moved.max()))
    r = load(folder, dtype, page_size=8)
    assert len(r.cache.kv_groups) == 1 and len(r.cache.kv_groups[0].entries) == 2
    for sizes in ([70], [1], [2], [33, 2, 1, 20]):
        assert_close(stepped(r, "x", toks, sizes), ref, dtype, f"readers, portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["sun_a", "sun_w"])
def test_long_decoding(tmp_path, name, dtype):
    """Four tokens of prompt and 200 decoded one by one through the decode graphs."""
    folder = make_nurasun_dir(tmp_path, name, fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    toks = steady_tokens(cfg, w, 204, 77)
    ref = reference(w, cfg, toks, dtype)
    r = load(folder, dtype, page_size=8)
    got = stepped(r, "long", toks, [4] + [1] * 200)
    assert r.graphs.replays >= 150
    assert_close(got, ref, dtype, "long decoding")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["sun_a", "sun_c"])
def test_greedy_generation_through_the_entry_point(tmp_path, name, dtype):
    """``Engine.run_offline``: scheduler, portions of prompts under a token budget, decode graphs, device sampling.
    Every generated token must be the plain model's choice (or tie with it within bfloat16's noise)."""
    from inf_engine_b200 import Engine, Request

    folder = make_nurasun_dir(tmp_path, name, fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    prompts = [random_tokens(cfg["vocab"], n, 60 + 100 * n) for n in (3, 41, 18, 1, 70)]
    outs = []
    for pipeline in (True, False):
        engine = Engine.from_dir(folder, dtype=dtype, n_total_blocks=24, block_size=8, max_requests=3,
                                 max_tokens_per_step=32, chunk=13, pipeline=pipeline)
        out = engine.run_offline([Request(i, p, max_new_tokens=10) for i, p in enumerate(prompts)])
        engine.runner.cache.check()
        assert engine.runner.cache.n_open == 0 and engine.runner.graphs.replays > 0
        outs.append(out)
        for i, p in enumerate(prompts):
            assert len(out[i]) == 10
            logits = plain.forward(cfg, w, p + out[i])
            for j, tok in enumerate(out[i]):
                row = logits[len(p) + j - 1]
                top = float(row.abs().max())
                slack = 1e-4 * top if dtype == "float32" else BF16_NEAR_TIE * NEAR_TIE_NOISE * max(1.0, top)
                assert float(row.max() - row[tok]) <= slack, f"{name} {dtype}: request {i}, token {j}"
    if dtype == "float32":
        assert outs[0] == outs[1]


def test_command_line_and_trace_replay(tmp_path):
    folder = make_nurasun_dir(tmp_path, "sun_b")
    cfg, w = plain_inputs(folder)
    prompt = random_tokens(cfg["vocab"], 12, 5)
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "generate_llama"), "--model-dir", str(folder),
                           "--prompt-ids", ",".join(map(str, prompt)), "--n", "6", "--dtype", "float32"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    ids = [int(t) for t in proc.stdout.strip().splitlines()[-1].split(": ")[1].split(",")]
    logits = plain.forward(cfg, w, prompt + ids)
    assert ids == [int(logits[len(prompt) + j - 1].argmax()) for j in range(6)]
    from test_gpu_replay import schedules
    for dtype in DTYPES:
        (tmp_path / dtype).mkdir()
        folder = make_nurasun_dir(tmp_path / dtype, "sun_b", fix=routers_for(dtype))
        cfg, w = plain_inputs(folder)
        requests = {str(i): steady_tokens(cfg, w, n, 300 + 50 * i) for i, n in enumerate([70, 45, 130, 20, 97, 33])}
        trace = schedules("sun", requests, seed=3)
        got = run_trace(folder, dtype, trace, tmp_path / f"out_{dtype}", cfg["vocab"], page_size=8)
        refs = {rid: reference(w, cfg, t, dtype) for rid, t in requests.items()}
        for prefix in "wdpm":
            for rid, t in requests.items():
                rows = [got.get((prefix + rid, p)) for p in range(len(t))]
                if rows[0] is None:
                    continue
                assert_close(torch.stack(rows), refs[rid], dtype, f"replay {prefix}{rid}")
