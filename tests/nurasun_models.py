"""Small Nurasun configurations for the tests, and model folders made from them.

They differ from one another in every size and constant: width, vocabulary, the residual's multiplier (and 1), the cap of
the logits (and none), head counts and groups (kv heads equal to the heads, one, a number in between), head sizes (most no
power of two, one odd), rotated dimensions (all, some, none), chunks (shorter than a page, no multiple of one, several
pages, none), compressed vectors of several sizes, latent layers that read another's vectors with other heads, head
sizes and scales (one reader, two readers of one layer, a reader several layers on), dense layers, mixtures with a shared
expert of the experts' size, of another size and without one, one or all experts a token, and layers without a
feed-forward.
"""

from __future__ import annotations

import json
from pathlib import Path

import torch


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _att(heads, kv, dim, scale, mlp, rot=None, chunk=None):
    """``rot`` (base, dims)."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _lat(heads, dim, vdim, rank, scale, mlp, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _model(vocab, width, eps, mult, cap, layers):
    out = {"architecture": "Nurasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}
    if cap is not None:
        out["logit_softcap"] = cap
    return out


# chunks that end inside a page; a latent layer, one that reads it across a layer between with other heads, a layer without
# a feed-forward, attention that neither rotates nor masks
SUN_A = _model(211, 60, 1e-5, 0.7, 2.5, [
    _att(4, 2, 16, 0.3, _dense(70), (300.0, 8), 20),
    _lat(3, 10, 6, 22, 0.35, _moe(6, 3, 28, 20)),
    _att(6, 3, 10, 0.4, None, None, None),
    _lat(5, 12, 14, 22, 0.3, _dense(44), 1),
])
# multiplier 1, no cap; a head a key head, everything rotated, chunks shorter than a page; two layers read one layer's
# vectors; a token runs every expert, no shared expert; a shared expert of the experts' size
SUN_B = _model(157, 96, 1e-6, 1.0, None, [
    _lat(4, 16, 16, 40, 0.25, _dense(50)),
    _att(3, 3, 24, 0.2, _moe(3, 3, 24), (1000.0, 24), 5),
    _lat(2, 24, 8, 40, 0.3, _moe(5, 2, 32, 32), 0),
    _lat(6, 8, 24, 40, 0.4, None, 0),
    _att(8, 4, 12, 0.3, _dense(36), (50.0, 12), 16),
])
# sizes that are multiples of nothing much: width 105, heads of 9, one key head under five, a compressed vector of 17
SUN_C = _model(131, 105, 0.03, 0.4, 6.0, [
    _att(5, 1, 9, 0.5, _moe(7, 1, 21, 33), (200.0, 6), 13),
    _lat(2, 7, 5, 17, 0.5, _dense(33)),
    _lat(3, 5, 9, 17, 0.6, _moe(2, 1, 19, 11), 1),
])
# sizes that the tensor-core attention takes, in prompts and decoding; four query heads a key head
SUN_W = _model(300, 128, 1e-5, 0.5, 10.0, [
    _att(8, 2, 32, 0.2, _dense(144), (10000.0, 16), 48),
    _lat(4, 32, 16, 64, 0.2, _moe(8, 3, 64, 128)),
    _lat(8, 16, 32, 64, 0.3, _dense(80), 1),
    _att(2, 2, 16, 0.3, _moe(8, 4, 32, 64), (500.0, 16), 100),
])
# heads of 64 that see every key, which the tcgen05 attention takes for portions of enough rows; widths that the tcgen05
# products take; 128 numbers a compressed vector
SUN_T = _model(200, 192, 1e-5, 0.6, 8.0, [
    _att(3, 1, 64, 0.13, _dense(128), (5000.0, 64)),
    _att(4, 2, 64, 0.15, _moe(4, 2, 64, 192), (5000.0, 32), 64),
    _lat(2, 64, 64, 128, 0.15, None),
    _lat(4, 32, 64, 128, 0.2, _moe(6, 2, 48, 64), 2),
])
# one mechanism each
SUN_ATT = _model(120, 48, 1e-5, 0.8, None, [_att(6, 3, 12, 0.4, None, (100.0, 8), 24)])
SUN_LAT = _model(120, 48, 1e-5, 0.8, None, [_lat(3, 12, 16, 24, 0.5, None), _lat(2, 16, 8, 24, 0.6, None, 0)])
SUN_MOE = _model(120, 48, 1e-6, 1.0, 3.0, [_att(1, 1, 16, 0.3, _moe(12, 4, 28, 40))])
SUN_DENSE = _model(120, 48, 1e-6, 0.5, 1.0, [_att(2, 2, 8, 0.3, _dense(40), (100.0, 4))])

MODELS = {"sun_a": SUN_A, "sun_b": SUN_B, "sun_c": SUN_C, "sun_w": SUN_W, "sun_t": SUN_T, "sun_att": SUN_ATT, "sun_lat": SUN_LAT,
          "sun_moe": SUN_MOE, "sun_dense": SUN_DENSE}
SEEDS = {name: 131 + i for i, name in enumerate(MODELS)}


def lively(tensors: dict) -> None:
    """Random tensors drawn N(0, std) leave some mechanisms almost idle; give them values that matter: a stream whose
    coordinates reach both the straight and the bent part of the hyperbolic tangent, offsets and biases of the size of what
    they are added to, activations of order one."""
    g = torch.Generator().manual_seed(29)
    for name, t in tensors.items():
        f = t.float()
        if name.endswith(".alpha"):
            f = 0.5 + torch.rand(f.shape, generator=g)
        elif name.endswith((".norm1", "final.norm")):
            f = 0.6 + 0.8 * torch.rand(f.shape, generator=g)
            f[::5] *= -1
        elif name.endswith(".norm"):
            f = 0.5 + torch.rand(f.shape, generator=g)
        elif name.endswith(("norm1.b", "final.norm.b")):
            f = 0.4 * torch.randn(f.shape, generator=g)
        elif name.endswith((".q.b", ".k.b")):
            f = 0.5 * torch.randn(f.shape, generator=g)
        elif name == "embed":
            f = f / f.std() * 0.8
        elif f.dim() == 2:                     # matrices by their fan-in, so that the stream stays of order one
            c = 1.5 if name.endswith((".mix.q", ".mix.k")) else (2.0 if name.endswith(".router") else 1.0)
            f = f / f.std() * c / f.shape[1] ** 0.5
        else:
            continue
        tensors[name] = f.to(t.dtype)


def make_nurasun_dir(tmp, name: str, store_dtype: str = "bfloat16", std: float = 0.08, fix=None, config: dict | None = None,
                     seed: int | None = None) -> Path:
    """A model folder with random weights for ``MODELS[name]`` (or ``config``); ``fix(tensors)`` may change them."""
    from inf_engine_b200.config import parse_config_dict
    from inf_engine_b200.parts import expected_tensors
    from inf_engine_b200.weights import random_tensors, write_safetensors

    d = config if config is not None else MODELS[name]
    out = Path(tmp) / f"{name}_{store_dtype}"
    out.mkdir(parents=True, exist_ok=True)
    cfg = parse_config_dict(d)
    tensors = random_tensors(expected_tensors(cfg.model_spec()), SEEDS.get(name, 7) if seed is None else seed, std=std,
                             store_dtype=store_dtype)
    lively(tensors)
    if fix is not None:
        fix(tensors)
    (out / "config.json").write_text(json.dumps(d, indent=1))
    write_safetensors(out / "model.safetensors", tensors, metadata={"format": "pt"})
    return out


def steady_routers(tensors: dict) -> None:
    """Routers that decide by a wide margin: the offset of a routed layer's norm gets a common direction, and the experts'
    rows lie along it at levels a step apart, over a small token-dependent part (the weights of the chosen experts still
    follow the token)."""
    g = torch.Generator().manual_seed(17)
    for name in list(tensors):
        if not name.endswith(".router"):
            continue
        b = name.replace("mlp.router", "norm1.b")
        common = torch.sign(torch.randn(tensors[b].shape[0], generator=g))
        tensors[b] = (tensors[b].float() * 0.5 + 0.6 * common).to(tensors[b].dtype)
        f = tensors[name].float()
        n = f.shape[0]
        level = (torch.arange(n, dtype=torch.float32)[torch.randperm(n, generator=g)] - n / 2) * 1.0
        tensors[name] = (0.04 * f + level[:, None] * common[None, :] / f.shape[1]).to(tensors[name].dtype)
