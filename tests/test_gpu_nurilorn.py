"""The Nurilorn family on the GPU against the plain implementation: each new kernel alone, each mechanism alone in a
small model, whole prompts against token-by-token decoding and portions down to two tokens, batches of unequal requests
with pages and state slots used again, the first tokens of a sequence, a far key that must stand out among hundreds in
every attention kernel, filters across the edges of portions and pages, long decoding, greedy generation through the
engine and its scheduler, the command line and the trace replay.  Every test runs in 32-bit and in bfloat16."""

import copy
import os
import random
import subprocess
import sys

import pytest
import torch

import plain_nurilorn as plain
from nurilorn_models import MODELS, _att, _dense, _model, _moe, make_nurilorn_dir, steady_routers
import helpers
from helpers import BF16_NEAR_TIE, plain_inputs, random_tokens, run_trace
from test_gpu_fovunex import F32_NOISE, NEAR_TIE_NOISE, close, dev_i32, k, load, stepped
from test_gpu_gavatar import CLOSE_CALL, GavRef

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F = torch.float64


def reference(w, cfg, toks, dtype):
    """The plain model's logits, for bfloat16 how far rounding alone moves each row, and which rows rest on no close call
    of a router (theirs and the rows whose filters reach back to one are left out of a comparison)."""
    gaps = []
    logits = plain.forward(cfg, w, toks, gaps=gaps)
    keep = torch.ones(len(toks), dtype=torch.bool)
    if gaps:
        ok = torch.stack(gaps).min(dim=0).values >= CLOSE_CALL[dtype]
        for back in range(4):
            keep[back:] &= ok[:len(ok) - back]
    if dtype == "float32":
        return GavRef(logits, None, keep)
    rounded = plain.forward(cfg, w, toks, round_to=torch.bfloat16)
    return GavRef(logits, (rounded - logits).norm(dim=-1) / logits.norm(dim=-1).clamp_min(1e-6), keep)


BF16_FLOOR = 0.006      # of a row's norm, beside three times what rounding alone moves the row


def assert_close(got, ref, dtype, what="", noise=1.0):
    got, want = got.double().cpu(), ref.logits
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    got, want = got[ref.keep], want[ref.keep]
    assert got.shape[0] >= max(1, ref.keep.numel() // 4), f"{what}: only {got.shape[0]} of {ref.keep.numel()} rows rest on no close call"
    if dtype == "float32":
        worst, tol = float((got - want).abs().max()), F32_NOISE * helpers.tolerance(dtype, want)
        helpers.STATS.append({"what": what, "dtype": dtype, "max_abs": worst, "tol": tol})
        assert worst <= tol, f"{what}: max |diff| {worst:.3e} > {tol:.3e}; worst row {int((got - want).abs().amax(-1).argmax())}"
        return
    rel = (got - want).norm(dim=-1) / want.norm(dim=-1).clamp_min(1e-6)
    bound = noise * (3.0 * ref.noise[ref.keep] + BF16_FLOOR)
    helpers.STATS.append({"what": what, "dtype": dtype, "rows": int(rel.numel()), "row_max": float(rel.max()),
                          "row_mean": float(rel.mean()), "worst_of_bound": float((rel / bound).max())})
    bad = (rel > bound).nonzero().flatten().tolist()
    assert not bad, (f"{what}: relative error of row {bad[0]} is {float(rel[bad[0]]):.3e} > {float(bound[bad[0]]):.3e}; rows over "
                     f"their bound: {bad[:20]} of {rel.numel()}; mean {float(rel.mean()):.3e}")


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
@pytest.mark.parametrize("d, groups, top", [(37, 1, 1), (60, 3, 1), (96, 2, 3), (100, 25, 2), (192, 4, 1), (105, 5, 4), (2048, 1, 2),
                                            (1536, 3, 4), (640, 16, 1), (64, 64, 1), (20480, 2, 1)])
def test_scaled_sum_with_the_grouped_norm_that_follows(dtype, d, groups, top):
    """residual += scale * y (or the weighted sum of several y) and the norm of the new rows, each part by itself; the sum
    alone; the norm alone; gathered rows, which leave the residual as it was."""
    dt = TORCH[dtype]
    g = torch.Generator().manual_seed(d + groups)
    n, eps = 6, 0.3
    res = torch.randn(n, d, generator=g) * (1 + 5 * torch.rand(n, d, generator=g))
    res[:, :d // groups] *= 20                              # one part far larger than the others
    scale, gain = torch.randn(d, generator=g), (1 + 0.5 * torch.randn(d, generator=g)).to(dt)
    for with_weights in ([False, True] if top == 1 else [True]):
        yt = torch.float32 if with_weights else dt
        pad = 0 if d % 4 == 0 and d > 64 else 3             # rows with and without a stride of their own
        y = torch.randn(n * top, d + pad, generator=g).to(yt)
        wts = torch.rand(n, top, generator=g) if with_weights else None
        yd = y.to(DEV)[:, :d]
        add = y.double()[:, :d]
        if with_weights:
            add = (add.reshape(n, top, d) * wts.double()[:, :, None]).sum(1)
        for sc in (scale, None):
            want_res = res.double() + (add * sc.double() if sc is not None else add)
            want = plain.group_norm(want_res, gain, groups, eps)
            args = (yd, sc.to(DEV) if sc is not None else None, wts.to(DEV) if with_weights else None)
            rd, out = res.to(DEV), torch.empty(n, d, dtype=dt, device=DEV)
            k().stream_norm(rd, *args, gain.to(DEV), groups, eps, out)
            assert torch.allclose(rd.double().cpu(), want_res, atol=1e-4, rtol=1e-5) and close(out, want, dtype, rel=1e-2)
            alone = res.to(DEV)
            k().stream_norm(alone, *args, None, 1, 0.0, None)
            assert torch.equal(alone, rd)
            rows = [4, 0, 4, 5]
            rd2, some = res.to(DEV), torch.empty(4, d, dtype=dt, device=DEV)
            k().stream_norm(rd2, *args, gain.to(DEV), groups, eps, some, row_index=dev_i32(rows))
            assert torch.equal(rd2.cpu(), res) and torch.equal(some, out[rows])
    rd, out = res.to(DEV), torch.empty(n, d, dtype=dt, device=DEV)
    k().stream_norm(rd, None, None, None, gain.to(DEV), groups, eps, out)
    assert torch.equal(rd.cpu(), res) and close(out, plain.group_norm(res.double(), gain, groups, eps), dtype, rel=1e-2)


def test_embedding_with_a_multiplier():
    table = torch.randn(11, 37).to(torch.bfloat16)
    ids = [3, 0, 10, 3]
    out = torch.empty(4, 37, dtype=torch.float32, device=DEV)
    k().embed_gather(dev_i32(ids), table.to(DEV), out, 2.7)
    assert torch.allclose(out.double().cpu(), table.double()[ids] * 2.7, rtol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv, hd, hdv, taps, rot, yarn, v_mode, halves", [
    (4, 2, 16, 24, 4, 8, (4.0, 32.0, 6.0, 0.5), None, False),     # sizes the 16-byte form takes in bfloat16
    (2, 2, 64, 64, 3, 64, None, "mix", False),
    (8, 2, 32, 16, 8, 12, None, "keep", False),                    # a rotation that ends inside a thread's eight channels
    (3, 3, 8, 8, 1, 8, None, "mix", False),
    (3, 1, 16, 8, 2, 0, None, "keep", False),
    (2, 1, 40, 8, 6, 2, None, None, False),
    (5, 1, 9, 5, 7, 6, (2.5, 20.0, 5.0, 0.7), "keep", False),      # sizes that only the other form takes: odd heads
    (3, 3, 12, 10, 4, 12, None, "mix", False),
    (2, 1, 16, 16, 16, 4, None, "mix", False),                     # sixteen taps
    (2, 2, 24, 8, 4, 8, None, "mix", True),                        # a rotation in halves
    (20, 4, 128, 256, 4, 128, None, "mix", False),                 # more channels than one block takes
    (3, 1, 8, 16, 0, 4, None, "mix", False),                       # no filters at all
])
def test_convolved_queries_keys_and_values(dtype, heads, kv, hd, hdv, taps, rot, yarn, v_mode, halves):
    """Three requests of unequal length in slots out of order: whole, and cut into portions down to one token with
    requests left out of a step; long enough that a request spans several of the kernel's chunks.  Padding tokens write
    nothing; the slot that nobody holds stays as it was."""
    dt = TORCH[dtype]
    g = torch.Generator().manual_seed(heads * 100 + hd)
    lens, slots, ps, lam = [75, 1, 22], [2, 0, 3], 8, 0.35
    qw, kw, vw = heads * hd, kv * hd, kv * hdv
    a8 = lambda n: -(-n // 8) * 8
    k0, v0 = a8(qw), a8(qw) + a8(kw)
    C = v0 + a8(vw)
    none = taps == 0
    taps = max(taps, 1)
    us = [torch.randn(L, C + 8, generator=g).to(dt) for L in lens]             # rows with a stride of their own
    wt = torch.randn(taps, C, generator=g) / taps ** 0.5
    if none:
        wt = None
    kept = [torch.randn(L, vw, generator=g).to(dt) for L in lens]
    rd = {"base": 300.0, "dims": rot}
    if yarn:
        rd["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    from inf_engine_b200.config import PositionSpec, YarnScaling
    from inf_engine_b200.parts.positions import partial_rotation_frequencies
    inv_freq, mult = None, 1.0
    if rot:
        inv_freq, mult = partial_rotation_frequencies(PositionSpec(kind="rotary_partial", theta=300.0, rot_dims=rot,
                                                                   yarn=YarnScaling(*yarn) if yarn else None))
        inv_freq = inv_freq.to(DEV)

    def turned(x):
        if not halves:
            return plain.rotate(x, rd)
        order = [i // 2 + (rot // 2 if i % 2 else 0) for i in range(rot)]        # halves: neighbour form of reordered dims
        y = x.clone()
        y[..., :rot] = x[..., order]
        y = plain.rotate(y, rd)
        out = y.clone()
        out[..., order] = y[..., :rot]
        return out

    wants = []
    for u, vk in zip(us, kept):
        T = u.shape[0]
        y = plain.causal_conv(u.double()[:, :C], wt.double().t()) if wt is not None else u.double()[:, :C]
        v = y[:, v0:v0 + vw]
        wants.append((turned(y[:, :qw].reshape(T, heads, hd)), turned(y[:, k0:k0 + kw].reshape(T, kv, hd)),
                      (1 - lam) * v + lam * vk.double() if v_mode == "mix" else v))

    def run(plan):
        state = torch.zeros(5, taps - 1, C, dtype=dt, device=DEV)
        state[1] = 7.0
        pages = sum(-(-L // ps) for L in lens) + 2
        kpool = torch.full((pages, kv, ps, hd), 9.0, dtype=dt, device=DEV)
        vpool = torch.full((pages, kv, ps, hdv), 9.0, dtype=dt, device=DEV)
        perm = torch.randperm(pages, generator=g).tolist()
        tables = [[perm.pop() for _ in range(-(-L // ps))] for L in lens]
        done, qs, vs = [0] * 3, [[] for _ in lens], [[] for _ in lens]
        for step in plan:
            reqs = [r for r in range(3) if step.get(r)]
            spans = [(r, done[r], done[r] + step[r]) for r in reqs]
            x = torch.cat([us[r][lo:hi] for r, lo, hi in spans]).to(DEV)
            n = x.shape[0]
            starts = [0]
            for _, lo, hi in spans:
                starts.append(starts[-1] + hi - lo)
            pos = [p for _, lo, hi in spans for p in range(lo, hi)]
            at = [tables[r][p // ps] * ps + p % ps for r, lo, hi in spans for p in range(lo, hi)]
            vk = torch.cat([kept[r][lo:hi] for r, lo, hi in spans]).to(DEV).contiguous()
            q = torch.empty(n, qw, dtype=dt, device=DEV)
            k().conv_qkv(x[:, :C], wt.to(DEV) if wt is not None else None, state, q, kpool, vpool, dev_i32(pos), dev_i32(at),
                         dev_i32(starts), dev_i32([slots[r] for r in reqs]), len(reqs), heads, kv, hd, hdv, k0, v0, ps,
                         inv_freq=inv_freq, rot_dims=rot, neighbours=not halves, mult=mult, v_kept=vk, v_mode=v_mode, lam=lam,
                         max_q_len=max(hi - lo for _, lo, hi in spans))
            for i, (r, lo, hi) in enumerate(spans):
                qs[r].append(q[starts[i]:starts[i + 1]].cpu())
                vs[r].append(vk[starts[i]:starts[i + 1]].cpu())
                done[r] = hi
        keys = [torch.stack([kpool[tables[r][p // ps], :, p % ps] for p in range(L)]).cpu() for r, L in enumerate(lens)]
        values = [torch.stack([vpool[tables[r][p // ps], :, p % ps] for p in range(L)]).cpu() for r, L in enumerate(lens)]
        used = int((kpool == 9.0).all(dim=-1).sum())
        assert used == kv * (pages * ps - sum(lens))                            # nothing beyond the tokens' own slots
        return [torch.cat(x) for x in qs], keys, values, [torch.cat(x) for x in vs], state.cpu()

    whole = run([{0: 75, 1: 1, 2: 22}])
    cut = run([{0: 5, 2: 1}, {0: 1, 1: 1}, {0: 34, 2: 3}, {2: 2, 0: 2}, {2: 16, 0: 1}, {0: 32}])
    for r, L in enumerate(lens):
        q, kk, v = wants[r]
        assert close(whole[0][r], q.reshape(L, qw), dtype, rel=1e-2) and close(whole[1][r], kk, dtype, rel=1e-2)
        assert close(whole[2][r], v.reshape(L, kv, hdv), dtype, rel=1e-2)
        for i in range(3):
            assert torch.equal(whole[i][r], cut[i][r]), (r, i)
        if v_mode == "keep":
            assert torch.equal(whole[3][r].reshape(L, kv, hdv), whole[2][r])
        for res in (whole, cut):
            if taps > 1:
                tail = torch.cat([torch.zeros(taps - 1, C, dtype=dt), us[r][:, :C]])[-(taps - 1):]
                for c0, width in ((0, qw), (k0, kw), (v0, vw)):
                    assert torch.equal(res[4][slots[r]][:, c0:c0 + width], tail[:, c0:c0 + width]), r
                assert bool((res[4][1] == 7.0).all())
    # padding: a request without a slot, tokens without a place
    state = torch.zeros(2, taps - 1, C, dtype=dt, device=DEV)
    kpool, vpool = (torch.full((2, kv, ps, x), 9.0, dtype=dt, device=DEV) for x in (hd, hdv))
    x = us[0][:2].to(DEV)
    q = torch.empty(2, qw, dtype=dt, device=DEV)
    k().conv_qkv(x[:, :C], wt.to(DEV) if wt is not None else None, state, q, kpool, vpool, dev_i32([0, 0]), dev_i32([-1, -1]),
                 dev_i32([0, 1, 2]), dev_i32([-1, -1]), 2, heads, kv, hd, hdv, k0, v0, ps, inv_freq=inv_freq, rot_dims=rot,
                 neighbours=not halves, mult=mult, max_q_len=1)
    assert bool((kpool == 9.0).all()) and bool((vpool == 9.0).all()) and (taps == 1 or float(state.abs().max()) == 0.0)


def test_router_of_softmax_scores_with_groups():
    """The softmax over all experts; groups by their largest score; ties to the lower index; weights over their sum."""
    for n_experts, top, count, keep in ((6, 3, 3, 2), (8, 3, 2, 1), (12, 4, 4, 2), (5, 5, 1, 1), (40, 6, 8, 3), (7, 1, 7, 2), (1, 1, 1, 1)):
        g = torch.Generator().manual_seed(n_experts)
        z = 2 * torch.randn(33, n_experts + 2, generator=g)
        z[0, :n_experts] = 1.0
        z[1, :n_experts] = torch.arange(n_experts) % 2
        z[2, :n_experts] *= 30                                   # scores that underflow
        ids = torch.empty(33, top, dtype=torch.int32, device=DEV)
        wts = torch.empty(33, top, dtype=torch.float32, device=DEV)
        k().moe_route(z.to(DEV)[:, :n_experts], None, ids, wts, None, n_experts, top, count, keep, 1.0, 1e-20, score="softmax",
                      group_score="max")
        for t in range(33):
            if t == 2:
                assert bool(torch.isfinite(wts[t]).all()) and float(wts[t].sum()) == pytest.approx(1.0, abs=1e-5)
                assert int(ids[t, 0]) == int(z[t, :n_experts].argmax())
                continue
            w = {"router": torch.eye(n_experts, dtype=F)}
            want, ww = plain.route(z[t:t + 1, :n_experts].double(), {"experts": n_experts, "top": top,
                                                                   "groups": {"count": count, "keep": keep}}, w, "")
            assert ids[t].tolist() == want[0], (n_experts, t)
            assert torch.allclose(wts[t].double().cpu(), torch.tensor(ww[0], dtype=F), atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, ff, experts, top, limit", [(40, 24, 5, 2, 0.8), (72, 20, 3, 1, 2.0), (64, 136, 4, 3, 1.1)])
def test_experts_with_clamped_branches(dtype, d, ff, experts, top, limit):
    """The grouped product with the clamped activation in its epilogue, on both of its kernels."""
    dt = TORCH[dtype]
    g = torch.Generator().manual_seed(d)
    n = 90
    x = (2 * torch.randn(n, d, generator=g)).to(dt)
    w = {}
    for e in range(experts):
        for name, shape in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))):
            w[f"e{e}.{name}"] = (torch.randn(shape, generator=g) / shape[1] ** 0.5).to(dt)
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(n)]).to(torch.int32)
    both = torch.stack([torch.stack([w[f"e{e}.gate"], w[f"e{e}.up"]], dim=1).reshape(2 * ff, d) for e in range(experts)]).contiguous()
    pairs = torch.empty(n * top, dtype=torch.int32, device=DEV)
    tiles = torch.empty(k().moe_max_tiles(n * top, experts), 4, dtype=torch.int32, device=DEV)
    k().moe_sort(ids.to(DEV), experts, pairs, tiles)
    hidden = torch.empty(n * top, ff, dtype=dt, device=DEV)
    k().moe_gemm(x.to(DEV), both.to(DEV), hidden, pairs, tiles, top, gather=True, scatter=False, epi="silu_mul", act=(1.702, limit, 1.0))
    got = torch.empty(n * top, ff, dtype=F)
    got[pairs.cpu().long()] = hidden.double().cpu()
    limits = 0
    for p in range(n * top):
        e, row = int(ids.reshape(-1)[p]), x.double()[p // top]
        a, b = w[f"e{e}.gate"].double() @ row, w[f"e{e}.up"].double() @ row
        limits += int((a > limit).sum()) + int((b.abs() > limit).sum())
        a, b = a.clamp(max=limit), b.clamp(-limit, limit)
        assert close(got[p], a * torch.sigmoid(1.702 * a) * (b + 1), dtype, rel=1e-2), p
    assert limits > 100


@pytest.mark.parametrize("kernel, n_heads, n_k, hd, hdv, cap", [
    (kernel, *shape) for kernel in ("rows", "general", "wide", "wide_small")
    for shape in ((8, 2, 16, 32, 7.0), (3, 3, 32, 16, 30.0), (4, 1, 48, 48, None), (6, 3, 64, 64, 2.5))] + [
    ("tcgen05", *shape) for shape in ((6, 3, 64, 64, 2.5), (8, 2, 64, 64, 30.0), (5, 5, 64, 64, None), (4, 1, 128, 128, 7.0),
                                      (3, 3, 128, 128, None))])
def test_a_far_key_stands_out_under_capped_scores(kernel, n_heads, n_k, hd, hdv, cap):
    """One key far back dominates every score it meets (its scores reach the cap); the denominator also holds the term of
    a score of 0, which is most of it for queries whose keys all score far below; every head passes its gate.  Unseen
    pages are poisoned.  float32 kernels in both storage types."""
    for dt in ([torch.bfloat16] if kernel.startswith(("wide", "tc")) else [torch.float32, torch.bfloat16]):
        g = torch.Generator().manual_seed(13)
        ps, T, scale, hot = 8, 331, 0.5, 37
        group = n_heads // n_k
        kk = torch.randn(T, n_k, hd, generator=g) * 0.3
        q = torch.randn(T, n_heads, hd, generator=g) * 0.3
        direction = torch.randn(hd, generator=g)
        direction /= direction.norm()
        kk[hot] += 25 * direction
        q += 2 * direction
        low = 200                                        # this query scores far below zero everywhere
        q[low] = -40 * direction
        kk[:hot] += 2 * direction
        kk[hot + 1:] += 2 * direction
        v = torch.randn(T, n_k, hdv, generator=g)
        gate = 2 * torch.randn(T, n_heads + 3, generator=g)
        kk, q, v, gate = kk.to(dt), q.to(dt), v.to(dt), gate.to(dt)
        n_pages = -(-T // ps)
        perm = torch.randperm(n_pages + 3, generator=g)[:n_pages]
        kpool = torch.full((n_pages + 3, n_k, ps, hd), float("nan"), dtype=dt)
        vpool = torch.full((n_pages + 3, n_k, ps, hdv), float("nan"), dtype=dt)
        for t in range(T):
            kpool[perm[t // ps], :, t % ps] = kk[t]
            vpool[perm[t // ps], :, t % ps] = v[t]
        rep = lambda x: x.double().repeat_interleave(group, dim=1)
        w = plain.weights(q.double(), rep(kk), scale, cap)
        want = torch.einsum("hij,jhd->ihd", w, rep(v)) * torch.sigmoid(gate.double()[:, :n_heads, None])
        wide = kernel.startswith("wide")
        small = kernel in ("rows", "wide_small")
        qpos = [hot - 1, hot, hot + 1, 63, 64, 65, 150, low, 201, 329, 7, 0] if small else list(range(30, T))
        out = torch.empty(len(qpos), n_heads * hdv, dtype=dt, device=DEV)
        qrows, gates = q[qpos].reshape(len(qpos), -1).to(DEV), gate[qpos].to(DEV)[:, :n_heads]
        extra = dict(v_head_dim=hdv, sink=torch.zeros(n_heads, device=DEV), softcap=cap or 0.0, gate=gates)
        table = perm.to(torch.int32)
        kp, vp = kpool.to(DEV), vpool.to(DEV)
        if small:
            R = len(qpos)
            tables = torch.stack([torch.where(torch.arange(n_pages) * ps <= p, table, -1) for p in qpos]).to(torch.int32)
            args = (qrows, out, kp, vp, tables.to(DEV), dev_i32(range(R + 1)), dev_i32(qpos), R, group, n_heads, n_k, hd, ps, None, scale)
            if kernel == "rows":
                k().attention_rows(*args, **extra)
            else:
                for splits in (1, None):
                    n_splits, split_keys = k().attention_wide_splits(hd, hdv, T + 64, R * n_k, capped=bool(cap))
                    if splits == 1:
                        n_splits, split_keys = 1, 0
                    words = k().attention_wide_small_scratch(hd, hdv, R, group, n_k, n_splits, capped=bool(cap))
                    scratch = torch.empty(max(words, 1), dtype=torch.float32, device=DEV)
                    k().attention_wide_small(*args, n_splits, split_keys, scratch, **extra)
                    assert close(out.reshape(R, n_heads, hdv), want[qpos], "bfloat16", rel=2e-2), (splits, n_splits)
        else:
            rows = {"wide": k().ATTENTION_WIDE_ROWS, "general": 32, "tcgen05": k().ATTENTION_TCGEN05_ROWS}[kernel]
            work = [(0, p0) for p0 in range(0, len(qpos) * group, rows)]
            fn = k().attention_wide if wide else k().attention_general
            if kernel == "tcgen05":
                assert k().attention_tcgen05_exact_supports(qrows, out, kp, vp, hd, hdv, ps, scale, cap or 0.0)
                extra.pop("v_head_dim")
                k().attention_tcgen05_exact(qrows, out, kp, vp, table[None].to(DEV), dev_i32([0, len(qpos)]), dev_i32([30]),
                                            dev_i32([x[0] for x in work]), dev_i32([x[1] for x in work]), len(work), n_heads, n_k,
                                            hd, ps, scale, **extra)
                assert k().attention_tcgen05_exact_error() == 0
            else:
                fn(qrows, out, kp, vp, table[None].to(DEV), dev_i32([0, len(qpos)]), dev_i32([30]), dev_i32([x[0] for x in work]),
                   dev_i32([x[1] for x in work]), len(work), n_heads, n_k, hd, ps, None, scale, **extra)
        got = out.double().cpu().reshape(len(qpos), n_heads, hdv)
        name = "float32" if dt is torch.float32 else "bfloat16"
        for i, p in enumerate(qpos):
            assert close(got[i], want[p], name, rel=2e-2), (kernel, dt, p, float((got[i] - want[p]).abs().max()))
        # the far key's weight is a real share where it is seen, and the low query leaves almost nothing
        assert float(w[:, 201, hot].min()) > (0.008 if cap == 2.5 else 0.3)
        assert float(w[:, low].sum(-1).max()) < (0.97 if cap == 2.5 else 0.5)


@pytest.mark.parametrize("kernel, hd", [("wide", 16), ("tcgen05", 64), ("tcgen05", 128), ("general", 16)])
def test_scores_up_to_the_cap_keep_float32_digits(kernel, hd):
    """The kernels' forms of the hyperbolic tangent against the exact one: n equal keys and values of 1, so that the
    output is the logistic of a score (plus ln n), over scores from tiny to far past the cap."""
    for cap in (0.5, 30.0, 60.0, 400.0):
        T, ps = 160, 16
        x = torch.linspace(-4, 4, T) * cap                       # the uncapped scores
        x[:64] = torch.linspace(-0.45, 0.45, 64) * cap           # a tile of queries far below the cap
        x[T // 2] = 1e-3 * cap
        q = torch.zeros(T, 1, hd)
        q[:, 0, 0] = x
        q = q.to(torch.bfloat16)
        kk = torch.zeros(T, 1, hd, dtype=torch.bfloat16)
        kk[:, 0, 0] = 1.0
        pool = lambda t: t.reshape(T // ps, 1, ps, hd).to(DEV)
        v = torch.ones(T, 1, hd, dtype=torch.bfloat16)
        out = torch.empty(T, hd, dtype=torch.bfloat16, device=DEV)
        rows = {"wide": k().ATTENTION_WIDE_ROWS, "general": 32, "tcgen05": k().ATTENTION_TCGEN05_ROWS}[kernel]
        work = list(range(0, T, rows))
        args = (q.reshape(T, hd).to(DEV), out, pool(kk), pool(v), dev_i32([list(range(T // ps))]), dev_i32([0, T]), dev_i32([0]),
                dev_i32([0] * len(work)), dev_i32(work), len(work), 1, 1, hd, ps)
        sink = torch.zeros(1, device=DEV)
        if kernel == "tcgen05":
            if cap > 60:
                assert not k().attention_tcgen05_exact_supports(args[0], out, args[2], args[3], hd, hd, ps, 1.0, cap)
                with pytest.raises(k().KernelError):
                    k().attention_tcgen05_exact(*args, 1.0, softcap=cap, sink=sink)
                continue
            k().attention_tcgen05_exact(*args, 1.0, softcap=cap, sink=sink)
            assert k().attention_tcgen05_exact_error() == 0
        else:
            (k().attention_wide if kernel == "wide" else k().attention_general)(*args, None, 1.0, softcap=cap, sink=sink)
        s = cap * torch.tanh(q[:, 0, 0].double() / cap)
        want = torch.sigmoid(s + torch.log(torch.arange(1, T + 1, dtype=F)))      # n equal scores s beside a score of 0
        assert torch.allclose(out[:, 0].double().cpu(), want, rtol=5e-3, atol=1e-30), (kernel, cap)


# =============================================================== whole models
LENGTH = {"nur_a": 97, "nur_b": 70, "nur_c": 131, "nur_w": 190, "nur_t": 280, "nur_att": 75, "nur_mix": 50, "nur_moe": 41, "nur_dense": 60}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_whole_prompt_decoding_and_portions_agree_with_the_plain_model(tmp_path, name, dtype):
    folder = make_nurilorn_dir(tmp_path, name, fix=routers_for(dtype))
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
def test_stream_after_every_layer(tmp_path, dtype):
    """The residual stream layer by layer, not the logits alone: the model is cut after 1, 2, .. layers."""
    folder = make_nurilorn_dir(tmp_path, "nur_a", fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    toks = steady_tokens(cfg, w, 33, 5)
    for n in range(1, len(cfg["layers"]) + 1):
        c = copy.deepcopy(MODELS["nur_a"])
        c["layers"] = c["layers"][:n]

        def fix(t):
            for name in list(t):
                if name in w:
                    t[name] = w[name].to(t[name].dtype)
        d = tmp_path / f"cut{n}"
        d.mkdir()
        part = make_nurilorn_dir(d, "nur_a", config=c, fix=fix)
        cc, ww = plain_inputs(part)
        r = load(part, dtype, page_size=8)
        assert_close(stepped(r, "x", toks, [33]), reference(ww, cc, toks, dtype), dtype, f"after {n} layers")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["nur_a", "nur_b", "nur_c", "nur_w", "nur_t"])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(tmp_path, name, dtype):
    """Seven requests, at most three live, portions of some beside decoded tokens of others, some left out of a step;
    the pool holds exactly what the fullest moment needs and free pages are filled with NaN."""
    from inf_engine_b200 import StepEntry

    folder = make_nurilorn_dir(tmp_path, name, fix=routers_for(dtype))
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
def test_first_tokens_of_a_sequence_and_a_slot_that_another_request_held(tmp_path, dtype):
    """Sequences of one, two and three tokens (shorter than the filters) in one batch; then new requests in the slots
    they held: the old requests' last inputs must not reach the new ones."""
    from inf_engine_b200 import StepEntry

    folder = make_nurilorn_dir(tmp_path, "nur_a", fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    r = load(folder, dtype, max_requests=3)
    first = {"a": steady_tokens(cfg, w, 1, 1), "b": steady_tokens(cfg, w, 2, 100), "c": steady_tokens(cfg, w, 3, 200)}
    for rid in first:
        r.open(rid)
    lg = r.step([StepEntry(rid, t, list(range(len(t)))) for rid, t in first.items()]).cpu()
    at = 0
    for rid, t in first.items():
        assert_close(lg[at:at + len(t)], reference(w, cfg, t, dtype), dtype, f"first tokens of {rid}")
        at += len(t)
    more = [9, 9, 120]
    for i, tok in enumerate(more):
        lg = r.step([StepEntry("b", [tok], [0])]).cpu()
        assert_close(lg, reference(w, cfg, first["b"] + more[:i + 1], dtype)[-1:], dtype, "second and later tokens")
    for rid in first:
        r.close(rid)
    second = {"d": steady_tokens(cfg, w, 9, 300), "e": steady_tokens(cfg, w, 1, 400), "f": steady_tokens(cfg, w, 2, 500)}
    for rid in second:
        r.open(rid)
    lg = r.step([StepEntry(rid, t, list(range(len(t)))) for rid, t in second.items()]).cpu()
    at = 0
    for rid, t in second.items():
        assert_close(lg[at:at + len(t)], reference(w, cfg, t, dtype), dtype, f"{rid} in a slot used before")
        at += len(t)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [2, 9])
def test_filters_across_the_edges_of_portions_and_pages(tmp_path, dtype, taps):
    """Filters whose oldest tap weighs most: a token shows the input exactly ``taps - 1`` places back and none further,
    whatever lies between them (a portion's edge, a page's edge, several portions of two tokens)."""
    config = _model(90, 48, 1e-5, 2, 2.0, 1.0, 1.0, [_att(3, 1, 16, 8, 0.4, taps, None, (100.0, 8), None, 8.0, True),
                                                     _att(2, 1, 8, 8, 0.4, taps, _dense(40, 1.5), None, None, None, True)])

    def fix(t):
        for name in list(t):
            if name.endswith(".conv"):
                f = 0.1 * t[name].float()
                f[:, 0] = 1.5
                t[name] = f.to(t[name].dtype)
    folder = make_nurilorn_dir(tmp_path, "taps", config=config, fix=fix)
    cfg, w = plain_inputs(folder)
    toks = steady_tokens(cfg, w, 45, 5)
    ref = reference(w, cfg, toks, dtype)
    w2 = {n: (torch.roll(t, 1, dims=1) if n.endswith(".conv") else t) for n, t in w.items()}    # a filter one place off
    wrong = plain.forward(cfg, w2, toks)
    assert float(((wrong - ref.logits).norm(dim=-1) / ref.logits.norm(dim=-1)).mean()) > 0.1
    r = load(folder, dtype, page_size=8)
    assert_close(stepped(r, "whole", toks, [45]), ref, dtype, f"{taps} taps: whole")
    assert_close(stepped(r, "decode", toks, [1] * 45), ref, dtype, f"{taps} taps: decoded")
    assert_close(stepped(r, "pairs", toks, [2]), ref, dtype, f"{taps} taps: portions of two")
    assert_close(stepped(r, "edges", toks, [taps - 1, taps, 8 - taps % 8, 1, taps + 1, 2]), ref, dtype, f"{taps} taps: edges")
    r.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["nur_att", "nur_w", "nur_t"])
def test_a_far_key_is_found(tmp_path, name, dtype):
    """The attention is made sharp; the test first shows that swapping one token 250 and more positions back moves the
    last positions' plain logits, then the engine must agree with the plain model there, in a prompt and decoded (the
    kernels alone are tested with a key that dominates)."""
    config = copy.deepcopy(MODELS[name])
    for L in config["layers"]:
        L["mixer"]["scale"] *= 2.0
    folder = make_nurilorn_dir(tmp_path, name, config=config, fix=routers_for(dtype) if name != "nur_att" else None)      # it has no router
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
@pytest.mark.parametrize("name", ["nur_a", "nur_w"])
def test_long_decoding(tmp_path, name, dtype):
    """Four tokens of prompt and 200 decoded one by one through the decode graphs."""
    folder = make_nurilorn_dir(tmp_path, name, fix=routers_for(dtype))
    cfg, w = plain_inputs(folder)
    toks = steady_tokens(cfg, w, 204, 77)
    ref = reference(w, cfg, toks, dtype)
    r = load(folder, dtype, page_size=8)
    got = stepped(r, "long", toks, [4] + [1] * 200)
    assert r.graphs.replays >= 150
    assert_close(got, ref, dtype, "long decoding")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["nur_a", "nur_c"])
def test_greedy_generation_through_the_entry_point(tmp_path, name, dtype):
    """``Engine.run_offline``: scheduler, portions of prompts under a token budget, decode graphs, device sampling.
    Every generated token must be the plain model's choice (or tie with it within bfloat16's noise)."""
    from inf_engine_b200 import Engine, Request

    folder = make_nurilorn_dir(tmp_path, name, fix=routers_for(dtype))
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
    folder = make_nurilorn_dir(tmp_path, "nur_b")
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
        folder = make_nurilorn_dir(tmp_path / dtype, "nur_b", fix=routers_for(dtype))
        cfg, w = plain_inputs(folder)
        requests = {str(i): steady_tokens(cfg, w, n, 300 + 50 * i) for i, n in enumerate([70, 45, 130, 20, 97, 33])}
        trace = schedules("nur", requests, seed=3)
        got = run_trace(folder, dtype, trace, tmp_path / f"out_{dtype}", cfg["vocab"], page_size=8)
        refs = {rid: reference(w, cfg, t, dtype) for rid, t in requests.items()}
        for prefix in "wdpm":
            for rid, t in requests.items():
                rows = [got.get((prefix + rid, p)) for p in range(len(t))]
                if rows[0] is None:
                    continue
                assert_close(torch.stack(rows), refs[rid], dtype, f"replay {prefix}{rid}")
