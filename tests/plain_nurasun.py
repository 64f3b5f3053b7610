"""A plain, slow Nurasun decoder in float64 on the CPU: whole sequences, no cache, one function per mechanism.

It shares no code with the package and is the oracle of the tests.  ``cfg`` is the ``config.json`` dictionary and
``w`` maps tensor names to torch tensors.  ``round_to`` (a torch dtype or None) rounds where an engine that keeps its
activations in that type rounds: what a norm hands to a product, the results of matrix products, and what is kept in
the cache; norms, angles, scores, softmax weights, the router and the residual stream stay float64 whatever it is.
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


def tanh_norm(x, w: dict, name: str):
    """tanh(alpha x) * gain + offset, coordinate by coordinate: nothing of the row's other coordinates enters."""
    alpha = w[name + ".alpha"].to(F).reshape(())
    return torch.tanh(alpha * x) * w[name].to(F) + w[name + ".b"].to(F)


def rms(x, gain, eps: float):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain.to(F)


def gelu(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, rot: dict | None):
    """x [T, heads, d]: dimension i of the first ``dims`` turns with i + dims / 2 by position * base^(-2 i / dims)."""
    dims = int(rot["dims"]) if rot else 0
    if not dims:
        return x
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=F)
    for i in range(dims // 2):
        a = (pos * float(rot["base"]) ** (-2.0 * i / dims))[:, None]
        u, v = x[:, :, i], x[:, :, i + dims // 2]
        out[:, :, i] = u * torch.cos(a) - v * torch.sin(a)
        out[:, :, i + dims // 2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def weights(q, k, scale: float, chunk: int | None = None):
    """Softmax weights [H, T, T] of every query over the keys at and before it, of its own chunk of positions only."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    T = s.shape[-1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    hidden = j > i
    if chunk:
        hidden = hidden | (torch.div(i, chunk, rounding_mode="floor") != torch.div(j, chunk, rounding_mode="floor"))
    return torch.softmax(s.masked_fill(hidden[None], float("-inf")), dim=-1)


def attention(h, m: dict, w: dict, p: str, round_to=None):
    """Rotated attention whose values are the projected keys before their rotation."""
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    G = int(m.get("kv_heads", H))
    q = lin(w[p + "q"], h) + w[p + "q.b"].to(F)
    k = lin(w[p + "k"], h) + w[p + "k.b"].to(F)
    q, k = rnd(q, round_to).reshape(T, H, d), rnd(k, round_to).reshape(T, G, d)
    v = k
    q, k = rnd(rotate(q, m.get("rot")), round_to), rnd(rotate(k, m.get("rot")), round_to)
    mask = m.get("mask")
    rep = H // G
    a = weights(q, k.repeat_interleave(rep, dim=1), float(m["scale"]), int(mask["size"]) if mask else None)
    o = rnd(torch.einsum("hij,jhd->ihd", a, v.repeat_interleave(rep, dim=1)), round_to)
    return lin(w[p + "o"], o.reshape(T, H * d), round_to)


def latent_vector(h, w: dict, p: str, eps: float, round_to=None):
    """The compressed vector of every token, as a cache holds it."""
    return rnd(rms(lin(w[p + "dkv"], h, round_to), w[p + "dkv.norm"], eps), round_to)


def latent_attention(h, c, m: dict, w: dict, p: str, round_to=None):
    """Attention without positions whose keys and values are expanded from the vectors ``c`` (this layer's or another's)."""
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    dv = int(m.get("vdim", d))
    q = lin(w[p + "q"], h, round_to).reshape(T, H, d)
    k, v = lin(w[p + "uk"], c).reshape(T, H, d), lin(w[p + "uv"], c).reshape(T, H, dv)
    a = weights(q, k, float(m["scale"]))
    o = rnd(torch.einsum("hij,jhd->ihd", a, v), round_to)
    return lin(w[p + "o"], o.reshape(T, H * dv), round_to)


def gated(h, w: dict, p: str, round_to=None):
    return lin(w[p + "down"], rnd(gelu(lin(w[p + "gate"], h)) * lin(w[p + "up"], h), round_to), round_to)


def squared_relu(h, w: dict, p: str, round_to=None, out_round=None):
    return lin(w[p + "down"], rnd(torch.relu(lin(w[p + "up"], h)) ** 2, round_to), out_round)


def route(h, r: dict, w: dict, p: str, gaps: list | None = None):
    """(chosen experts, their weights), a list a token.  ``gaps`` takes how close the choice was, in units of the
    logits' spread."""
    z = lin(w[p + "router"], h)
    s = torch.sigmoid(z)
    E, top = int(r["experts"]), int(r["top"])
    ids, wts, gap = [], [], []
    for t in range(h.shape[0]):
        row = s[t].tolist()
        order = sorted(range(E), key=lambda e: (-row[e], e))
        ids.append(order[:top])
        total = sum(row[e] for e in order[:top]) + 1e-20
        wts.append([row[e] / total for e in order[:top]])
        gap.append(float(z[t][order[top - 1]] - z[t][order[top]]) / max(float(z[t].std()), 1e-12) if top < E else float("inf"))
    if gaps is not None:
        gaps.append(torch.tensor(gap, dtype=F))
    return ids, wts


def mixture(h, mlp: dict, w: dict, p: str, round_to=None, gaps: list | None = None):
    ids, wts = route(h, mlp["router"], w, p, gaps)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t], wts[t]):
            out[t] += a * squared_relu(h[t:t + 1], w, f"{p}e{e}.", round_to)[0]
    if mlp.get("shared"):
        out = out + squared_relu(h, w, p + "shared.", round_to, round_to)
    return out


def forward(cfg: dict, w: dict, tokens: list[int], round_to=None, collect: list | None = None,
            gaps: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence; ``collect`` takes the residual stream after every layer, ``gaps`` the
    routers' margins (see ``route``)."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = w["embed"].to(F)[torch.tensor(tokens)]
    latents: dict = {}
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        h = rnd(tanh_norm(x, w, p + "norm1"), round_to)
        if L["type"] == "attention":
            y = attention(h, m, w, p + "mix.", round_to)
        else:
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent_vector(h, w, p + "mix.", eps, round_to)
            y = latent_attention(h, latents[i if src is None else int(src)], m, w, p + "mix.", round_to)
        if mlp is not None:
            y = y + (gated(h, w, p + "mlp.", round_to) if mlp["kind"] == "dense" else mixture(h, mlp, w, p + "mlp.", round_to, gaps))
        x = x + mult * y
        if collect is not None:
            collect.append(x.clone())
    logits = lin(w["head"], rnd(tanh_norm(x, w, "final.norm"), round_to))
    cap = cfg.get("logit_softcap")
    return float(cap) * torch.tanh(logits / float(cap)) if cap else logits


def forward_float32(cfg: dict, w: dict, tokens: list[int]) -> torch.Tensor:
    """The same model with every number a 32-bit float (how far 32-bit arithmetic alone moves the logits)."""
    global F
    F = torch.float32
    try:
        return forward(cfg, w, tokens).double()
    finally:
        F = torch.float64
