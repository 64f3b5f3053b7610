"""A plain, slow Nurilorn decoder in float64 on the CPU: whole sequences, no cache, one function per mechanism.

It shares no code with the package and is the oracle of the tests.  ``cfg`` is the ``config.json`` dictionary and
``w`` maps tensor names to torch tensors.  ``round_to`` (a torch dtype or None) rounds where an engine that keeps its
activations in that type rounds: what a norm hands to a product, the results of matrix products and convolutions, and
what is kept in the cache; norms, angles, scores, softmax weights, the router, every gate and the residual stream stay
float64 whatever it is.
"""

from __future__ import annotations

import math

import torch

F = torch.float64


def rnd(x: torch.Tensor, round_to) -> torch.Tensor:
    return x if round_to is None else x.to(round_to).to(F)


def lin(w: torch.Tensor, x: torch.Tensor, round_to=None) -> torch.Tensor:
    """W x for every row of x; W is stored [out, in]."""
    return rnd(x @ w.to(F).t(), round_to)


def group_norm(x, g, groups: int, eps: float):
    """RMS norm of each of ``groups`` equal consecutive parts by itself; the whole times g."""
    T, d = x.shape
    parts = x.reshape(T, groups, d // groups)
    out = torch.empty_like(parts)
    for j in range(groups):
        part = parts[:, j]
        out[:, j] = part / torch.sqrt((part ** 2).sum(-1, keepdim=True) / part.shape[-1] + eps)
    return out.reshape(T, d) * g.to(F)


def causal_conv(u, weight, round_to=None):
    """y_t = sum_j weight[:, j] u_(t - taps + 1 + j), with zeros before the start; a filter per channel."""
    T, taps = u.shape[0], weight.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += weight[:, j].to(F) * u[s]
    return rnd(y, round_to)


def frequencies(rot: dict) -> tuple[list[float], float]:
    """Frequencies of the rotated pairs, and the multiplier of sine and cosine."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    factor, original = float(s["factor"]), float(s["original"])

    def pair_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(pair_of(float(s["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(s["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, rot: dict | None):
    """x [T, heads, d]: neighbours (2i, 2i + 1) of the first dims turn by position * f_i, the rest passes."""
    if not rot or not int(rot.get("dims", 0)):
        return x
    f, mult = frequencies(rot)
    x = x.clone()
    pos = torch.arange(x.shape[0], dtype=F)
    for i, fi in enumerate(f):
        c, s = (torch.cos(pos * fi) * mult)[:, None], (torch.sin(pos * fi) * mult)[:, None]
        u, v = x[:, :, 2 * i].clone(), x[:, :, 2 * i + 1].clone()
        x[:, :, 2 * i], x[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return x


def weights(q, k, scale: float, softcap: float | None, sink: bool = True):
    """Causal weights [H, T, T]: exp(s) / (1 + sum exp(s)) with s = cap tanh(q . k scale / cap)."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    T = s.shape[-1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    s = s.masked_fill((j > i)[None], float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink:
        top = top.clamp_min(0.0)
    e = torch.exp(s - top)
    below = e.sum(-1, keepdim=True)
    return e / (below + torch.exp(-top) if sink else below)


def attention(h, m: dict, w: dict, p: str, round_to=None, first_v: dict | None = None):
    """``first_v`` carries the values of the first layer that mixes values to the later ones."""
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    G, dv = int(m.get("kv_heads", H)), int(m.get("vdim", d))

    def branch(name):
        u = lin(w[p + name], h, round_to)
        return causal_conv(u, w[p + name + ".conv"], round_to) if p + name + ".conv" in w else u

    q, k, v = branch("q").reshape(T, H, d), branch("k").reshape(T, G, d), branch("v").reshape(T, G, dv)
    q, k = rnd(rotate(q, m.get("rot")), round_to), rnd(rotate(k, m.get("rot")), round_to)
    if m.get("v_mix"):
        if "v" not in first_v:
            first_v["v"] = v.reshape(T, G * dv)
        else:
            lam = w[p + "vmix"].to(F).reshape(())
            v = rnd((1 - lam) * v + lam * first_v["v"].reshape(T, G, dv), round_to)
    rep = H // G
    a = weights(q, k.repeat_interleave(rep, dim=1), float(m["scale"]), m.get("softcap"))
    o = rnd(torch.einsum("hij,jhd->ihd", a, v.repeat_interleave(rep, dim=1)), round_to)
    o = rnd(o * torch.sigmoid(lin(w[p + "g"], h, round_to))[:, :, None], round_to)
    return lin(w[p + "o"], o.reshape(T, H * dv), round_to)


def feed_forward(x, w: dict, p: str, limit: float, round_to=None, out_round=None):
    g = torch.clamp(lin(w[p + "gate"], x), max=limit)
    u = torch.clamp(lin(w[p + "up"], x), -limit, limit)
    return lin(w[p + "down"], rnd(g * torch.sigmoid(1.702 * g) * (u + 1), round_to), out_round)


def route(h, r: dict, w: dict, p: str, gaps: list | None = None):
    """(chosen experts, their weights), a list a token.  ``gaps`` takes how close the choice was, in units of the
    scores' spread (over groups and over experts)."""
    z = lin(w[p + "router"], h)
    s = torch.softmax(z, dim=-1)
    E, top = int(r["experts"]), int(r["top"])
    grp = r.get("groups") or {}
    n, keep = int(grp.get("count", 1)), int(grp.get("keep", grp.get("count", 1)))
    per = E // n
    ids, wts, gap = [], [], []
    for t in range(h.shape[0]):
        row = s[t].tolist()
        best = sorted(range(n), key=lambda g: -max(row[g * per:(g + 1) * per]))
        allowed = [e for g in best[:keep] for e in range(g * per, (g + 1) * per)]
        order = sorted(allowed, key=lambda e: (-row[e], e))
        ids.append(order[:top])
        total = sum(row[e] for e in order[:top]) + 1e-20
        wts.append([row[e] / total for e in order[:top]])
        lg = z[t]
        close = []
        if keep < n:
            close.append(float(lg[best[keep - 1] * per:(best[keep - 1] + 1) * per].max() - lg[best[keep] * per:(best[keep] + 1) * per].max()))
        if top < len(order):
            close.append(float(lg[order[top - 1]] - lg[order[top]]))
        gap.append(min(close) / max(float(lg.std()), 1e-12) if close else float("inf"))
    if gaps is not None:
        gaps.append(torch.tensor(gap, dtype=F))
    return ids, wts


def mixture(h, mlp: dict, w: dict, p: str, round_to=None, gaps: list | None = None):
    ids, wts = route(h, mlp["router"], w, p, gaps)
    limit = float(mlp["expert"]["limit"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t], wts[t]):
            out[t] += a * feed_forward(h[t:t + 1], w, f"{p}e{e}.", limit, round_to)[0]
    return out


def forward(cfg: dict, w: dict, tokens: list[int], round_to=None, collect: list | None = None,
            gaps: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence; ``collect`` takes the residual stream after every layer, ``gaps`` the
    routers' margins (see ``route``)."""
    eps, groups = float(cfg["norm"]["eps"]), int(cfg["norm"].get("groups", 1))
    m = float(cfg.get("residual_mult", 1.0))
    x = w["embed"].to(F)[torch.tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    first_v: dict = {}
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rnd(group_norm(x, w[p + "norm1"], groups, eps), round_to)
        x = x + m * w[p + "ls1"].to(F) * attention(h, L["mixer"], w, p + "mix.", round_to, first_v)
        mlp = L.get("mlp")
        if mlp is not None:
            h = rnd(group_norm(x, w[p + "norm2"], groups, eps), round_to)
            if mlp["kind"] == "dense":
                y = feed_forward(h, w, p + "mlp.", float(mlp["limit"]), round_to, round_to)
            else:
                y = mixture(h, mlp, w, p + "mlp.", round_to, gaps)
            x = x + m * w[p + "ls2"].to(F) * y
        if collect is not None:
            collect.append(x.clone())
    h = rnd(group_norm(x, w["final.norm"], groups, eps), round_to)
    return lin(w["head"], h) * float(cfg.get("logit_scale", 1.0))


def forward_float32(cfg: dict, w: dict, tokens: list[int]) -> torch.Tensor:
    """The same model with every number a 32-bit float (how far 32-bit arithmetic alone moves the logits)."""
    global F
    F = torch.float32
    try:
        return forward(cfg, w, tokens).double()
    finally:
        F = torch.float64
