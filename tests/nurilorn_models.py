"""Small Nurilorn configurations for the tests, and model folders made from them.

They differ from one another in every size and constant: width, vocabulary, norm groups (one, some), the three constant
multipliers (and all of them 1), head counts and groups (kv heads equal to the heads, one, a number in between), key and
value head sizes (equal and unequal, most no power of two, one odd), rotated dimensions (all, some, none) with and
without blended frequencies, taps (none, one, more tokens than a page holds), capped scores or not, which layers mix
values (the first such layer first, in the middle, none), limits of the activation, dense layers, mixtures with one
group, several, as many groups as experts, one or all experts a token, and layers without a feed-forward.
"""

from __future__ import annotations

import json
from pathlib import Path

import torch


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, count, keep, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def _att(heads, kv, dim, vdim, scale, conv, mlp, rot=None, yarn=None, softcap=None, v_mix=False):
    """``rot`` (base, dims); ``yarn`` (factor, original, fast, slow)."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if conv:
        m["conv"] = conv
    if softcap is not None:
        m["softcap"] = softcap
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if yarn is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _model(vocab, width, eps, groups, scale, mult, logit, layers):
    return {"architecture": "Nurilorn", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
            "embedding": {"scale": scale}, "residual_mult": mult, "logit_scale": logit, "layers": layers}


# three norm groups; values mixed over layers of other head counts and sizes (two heads of 24, three of 16) with a layer
# in between that mixes none, has no rotation, no cap and no feed-forward
NUR_A = _model(211, 60, 1e-5, 3, 5.0, 0.7, 0.4, [
    _att(4, 2, 16, 24, 0.3, 4, _dense(70, 1.1), (300.0, 8), (4.0, 32.0, 6.0, 0.5), 9.0, True),
    _att(5, 1, 12, 8, 0.35, 2, None),
    _att(6, 3, 10, 16, 0.4, 3, _moe(6, 3, 3, 2, 28, 0.8), (500.0, 10), None, 4.0, True),
    _att(2, 2, 8, 24, 0.35, 5, _moe(4, 1, 2, 1, 40, 0.9), (80.0, 4), (2.0, 16.0, 4.0, 1.0), None, True),
])
# every multiplier 1 and one norm group; the first layer that mixes values is the second; filters of one tap and none at
# all; as many groups as experts; a token runs every expert
NUR_B = _model(157, 96, 1e-6, 1, 1.0, 1.0, 1.0, [
    _att(3, 3, 24, 24, 0.2, 1, _moe(5, 2, 5, 3, 36, 1.3), (1000.0, 24), None, 20.0, False),
    _att(4, 4, 12, 12, 0.3, 0, _moe(3, 3, 1, 1, 24, 0.7), (50.0, 6), (3.0, 24.0, 6.0, 0.5), 6.0, True),
    _att(8, 4, 12, 12, 0.3, 3, _dense(50, 2.0), (50.0, 12), None, None, True),
])
# sizes that are multiples of nothing much: width 105 in five groups, heads of 9 and 5, one kv head under five, seven taps
NUR_C = _model(131, 105, 1e-5, 5, 0.6, 1.4, 2.5, [
    _att(5, 1, 9, 5, 0.5, 7, _moe(7, 3, 1, 1, 20, 1.2), (200.0, 6), (2.5, 20.0, 5.0, 0.7), 3.0, True),
    _att(2, 1, 10, 5, 0.5, 7, _dense(33, 0.6), (200.0, 2), None, 5.0, True),
])
# head sizes that are multiples of 16, which the tensor-core attention of prompt portions takes; four query heads a key
# head, which send decode tokens there too; then one query head a key head
NUR_W = _model(300, 128, 1e-5, 4, 3.0, 0.6, 0.3, [
    _att(8, 2, 32, 16, 0.2, 4, _dense(144, 1.4), (10000.0, 16), (8.0, 64.0, 16.0, 1.0), 12.0, True),
    _att(2, 2, 64, 16, 0.15, 4, _moe(8, 3, 4, 2, 64, 1.1), (10000.0, 64), None, 15.0, True),
    _att(4, 1, 16, 32, 0.3, 2, _moe(8, 4, 2, 2, 32, 0.9), (10000.0, 8), None, None, True),
])
# heads of 64, which the tcgen05 attention takes for portions of enough rows: three query heads a key head under a cap; no
# cap, a head a key head; a cap beyond what its fixed reference allows, which sends the layer to the other kernels
NUR_T = _model(200, 144, 1e-5, 2, 2.0, 0.7, 0.5, [
    _att(3, 1, 64, 64, 0.13, 3, _dense(80, 1.4), (5000.0, 32), (4.0, 64.0, 16.0, 1.0), 25.0, True),
    _att(2, 1, 64, 64, 0.2, 4, None, (5000.0, 20), None, None, True),
    _att(1, 1, 64, 64, 0.2, 4, _moe(4, 2, 2, 1, 48, 1.0), None, None, 90.0, True),
])
# one mechanism each
NUR_ATT = _model(120, 48, 1e-5, 2, 2.0, 0.8, 1.0, [_att(6, 3, 12, 8, 0.4, 4, None, (100.0, 8), None, 5.0)])
NUR_MIX = _model(120, 48, 1e-5, 1, 2.0, 1.0, 1.0, [_att(3, 3, 8, 16, 0.4, 0, None, None, None, None, True) for _ in range(3)])
NUR_MOE = _model(120, 48, 1e-6, 1, 2.0, 1.0, 1.0, [_att(1, 1, 16, 16, 0.3, 0, _moe(12, 4, 4, 2, 28, 1.0))])
NUR_DENSE = _model(120, 48, 1e-6, 6, 2.0, 0.5, 2.0, [_att(2, 2, 8, 8, 0.3, 2, _dense(40, 0.5), (100.0, 4))])

MODELS = {"nur_a": NUR_A, "nur_b": NUR_B, "nur_c": NUR_C, "nur_w": NUR_W, "nur_t": NUR_T, "nur_att": NUR_ATT, "nur_mix": NUR_MIX,
          "nur_moe": NUR_MOE, "nur_dense": NUR_DENSE}
SEEDS = {name: 81 + i for i, name in enumerate(MODELS)}


def lively(tensors: dict) -> None:
    """Random tensors drawn N(0, std) leave some mechanisms almost idle; give them values that matter: norm and layer
    scales away from one (some negative), filters whose older taps weigh as much as the newest, shares of kept values
    from none to more than all, gates from shut to open, activations that reach their limits."""
    g = torch.Generator().manual_seed(83)
    for name, t in tensors.items():
        f = t.float()
        if name.endswith((".norm1", ".norm2")) or name == "final.norm":
            f = 0.6 + 0.8 * torch.rand(f.shape, generator=g)
        elif name.endswith((".ls1", ".ls2")):
            f = 0.2 + torch.rand(f.shape, generator=g)
            f[::7] *= -1
        elif name.endswith(".conv"):
            f = torch.randn(f.shape, generator=g) / f.shape[1] ** 0.5
        elif name.endswith(".vmix"):
            f = 0.2 + 0.6 * torch.rand(f.shape, generator=g)
        elif name.endswith((".mix.q", ".mix.k", ".mix.g", ".router", ".gate", ".up")):
            f = f * 3
        elif name == "embed":
            f = f * 4
        else:
            continue
        tensors[name] = f.to(t.dtype)


def make_nurilorn_dir(tmp, name: str, store_dtype: str = "bfloat16", std: float = 0.08, fix=None, config: dict | None = None,
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
    for i, L in enumerate(d["layers"]):          # the first mixing layer's own share is in the file and idle
        if L["mixer"].get("v_mix") and f"l{i}.mix.vmix" not in tensors:
            tensors[f"l{i}.mix.vmix"] = torch.tensor(0.9).to(tensors["embed"].dtype)
    if fix is not None:
        fix(tensors)
    (out / "config.json").write_text(json.dumps(d, indent=1))
    write_safetensors(out / "model.safetensors", tensors, metadata={"format": "pt"})
    return out


def steady_routers(tensors: dict) -> None:
    """Routers that decide by a wide margin: every embedding row gets a common component that survives the norms, and the
    experts' rows lie along it at levels a step apart, over a small token-dependent part (the weights of the chosen
    experts still follow the token)."""
    g = torch.Generator().manual_seed(17)
    embed = tensors["embed"].float()
    common = torch.sign(torch.randn(embed.shape[1], generator=g)) * embed.std() * 1.5
    tensors["embed"] = (embed + common).to(tensors["embed"].dtype)
    for name in list(tensors):
        if name.endswith(".router"):
            f = tensors[name].float()
            n = f.shape[0]
            level = (torch.arange(n, dtype=torch.float32)[torch.randperm(n, generator=g)] - n / 2) * 0.5
            f = 0.02 * f + level[:, None] * torch.sign(common)[None, :] / f.shape[1]
            tensors[name] = f.to(tensors[name].dtype)
        elif name.endswith((".ls1", ".ls2")):
            tensors[name] = (0.5 * tensors[name].float()).to(tensors[name].dtype)
