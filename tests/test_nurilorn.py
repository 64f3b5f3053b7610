"""The Nurilorn family without a GPU: configuration and its errors, the tensor table, the cache groups its layers ask
for, and the plain implementation's own consistency (grouped norm, convolution, blended frequencies, capped scores and
the denominator's constant, mixed values, the router), each by hand on small numbers."""

import copy
import math

import pytest
import torch

import plain_nurilorn as plain
from nurilorn_models import MODELS, make_nurilorn_dir
from helpers import plain_inputs, random_tokens

from inf_engine_b200.cache.manager import CacheManager, CacheRequirement
from inf_engine_b200.config import ConfigError, NurilornConfig, parse_config_dict
from inf_engine_b200.parts import expected_tensors

F = torch.float64


def test_config_round_trip_and_specs():
    for name, d in MODELS.items():
        cfg = parse_config_dict(d)
        assert isinstance(cfg, NurilornConfig)
        assert cfg.to_hf_dict() == d, name
        spec = cfg.model_spec()
        assert spec.kind == "decoder" and spec.head == "head" and spec.embedding_scale == d["embedding"]["scale"]
        assert spec.final_norm.groups == d["norm"]["groups"] and spec.final_norm.out_scale == d["logit_scale"]
        mixing = [i for i, L in enumerate(d["layers"]) if L["mixer"]["v_mix"]]
        for i, (blk, L) in enumerate(zip(spec.layers, d["layers"])):
            m = L["mixer"]
            assert blk.kind == "scaled_prenorm" and blk.residual_mult == d["residual_mult"]
            assert blk.mixer_norm.kind == "grouped_rmsnorm" and blk.mixer_norm.out_scale == 1.0
            assert (blk.feedforward is None) == (L["mlp"] is None)
            assert blk.mixer.softcap == m.get("softcap") and blk.mixer.sink == 0.0
            assert blk.mixer.v_keep == (mixing[:1] == [i])
            assert blk.mixer.v_mix == (f"l{i}.mix.vmix" if i in mixing[1:] else None)
            assert (blk.mixer.q_conv is None) == ("conv" not in m)
            assert blk.mixer.position.kind == ("rotary_partial" if "rot" in m else "none")
            if L["mlp"] is not None:
                assert blk.feedforward.activation == "clamped_swish" and blk.feedforward.up_offset == 1.0
            if L["mlp"] is not None and L["mlp"]["kind"] == "moe":
                assert blk.feedforward.score == "softmax" and blk.feedforward.group_score == "max"
                assert blk.feedforward.act_limit == L["mlp"]["expert"]["limit"]


def test_what_the_file_may_leave_out():
    d = {"architecture": "Nurilorn", "vocab": 50, "width": 24, "norm": {"eps": 1e-5},
         "layers": [{"type": "attention", "mixer": {"heads": 2, "dim": 9, "rot": None, "softcap": None}, "mlp": None},
                    {"type": "attention", "mixer": {"heads": 2, "dim": 8, "rot": {"base": 10.0, "scaling": None}},
                     "mlp": {"kind": "moe", "expert": {"ff": 8, "limit": 1}, "router": {"experts": 3, "top": 2}}}]}
    cfg = parse_config_dict(d)
    assert cfg.norm_groups == 1 and cfg.embedding_scale == cfg.residual_mult == cfg.logit_scale == 1.0
    a, b = cfg.layers
    assert a.mixer.kv_heads == 2 and a.mixer.vdim == 9 and a.mixer.scale == pytest.approx(1 / 3) and a.mixer.rot is None
    assert a.mixer.conv == 0 and a.mixer.softcap is None and not a.mixer.v_mix
    assert b.mixer.rot.dims == 8 and b.mixer.rot.yarn is None and (b.mlp.groups, b.mlp.keep_groups) == (1, 1)


def test_tensor_table():
    t = expected_tensors(parse_config_dict(MODELS["nur_a"]).model_spec())
    assert t["embed"].shape == (211, 60) and t["head"].shape == (211, 60)
    for n in ("l0.norm1", "l0.norm2", "l0.ls1", "l0.ls2", "l1.norm1", "l1.ls1", "final.norm"):
        assert t[n].shape == (60,), n
    assert t["l0.mix.q"].shape == (64, 60) and t["l0.mix.k"].shape == (32, 60) and t["l0.mix.v"].shape == (48, 60)
    assert t["l0.mix.q.conv"].shape == (64, 4) and t["l2.mix.v.conv"].shape == (48, 3)
    assert t["l0.mix.g"].shape == (4, 60) and t["l0.mix.o"].shape == (60, 96)
    assert "l0.mix.vmix" not in t and "l1.mix.vmix" not in t and t["l2.mix.vmix"].shape == () and t["l3.mix.vmix"].shape == ()
    assert t["l0.mlp.gate"].shape == (70, 60) and t["l0.mlp.down"].shape == (60, 70)
    assert "l1.norm2" not in t and "l1.ls2" not in t
    assert t["l2.mlp.router"].shape == (6, 60) and t["l2.mlp.e5.up"].shape == (28, 60) and "l2.mlp.e6.up" not in t
    spec = parse_config_dict(MODELS["nur_a"]).model_spec()
    assert {"l0.mix.vmix", "l1.mix.vmix", "l1.norm2", "l1.ls2"} <= set(spec.optional_tensors)
    assert "l1.mix.q.conv" not in expected_tensors(parse_config_dict(MODELS["nur_b"]).model_spec())


@pytest.mark.parametrize("change, text", [
    (lambda d: d["layers"][0].update(type="mlstm"), "not built"),
    (lambda d: d["layers"][0]["mlp"].update(kind="conv"), "not built"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda d: d["layers"][2]["mlp"]["router"].update(top=5), "cannot be chosen"),
    (lambda d: d["layers"][2]["mlp"]["router"]["groups"].update(count=4), "equal groups"),
    (lambda d: d["layers"][2]["mlp"]["router"]["groups"].update(keep=4), "cannot be kept"),
    (lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][0]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda d: d["layers"][2]["mixer"].update(vdim=8), "values a token"),
    (lambda d: d["norm"].update(groups=7), "norm groups"),
    (lambda d: d.pop("width"), "width"),
])
def test_config_errors(change, text):
    d = copy.deepcopy(MODELS["nur_a"])
    change(d)
    with pytest.raises(ConfigError, match=text):
        parse_config_dict(d)


def test_cache_groups_of_the_layers():
    pages = lambda g, d, dv: CacheRequirement(kind="kv", n_kv_heads=g, head_dim=d, v_head_dim=dv, dtype=torch.float32)
    inputs = lambda taps, c: CacheRequirement(kind="state", state_shape=(taps - 1, c), state_dtype=torch.float32)
    runs = [CacheRequirement(kind="several", parts=(pages(2, 16, 24), inputs(4, 144))), pages(4, 12, 12),
            CacheRequirement(kind="several", parts=(pages(2, 16, 24), inputs(4, 144)))]
    m = CacheManager(runs, page_size=8, n_pages=10, max_requests=2)
    assert len(m.kv_groups) == 2 and len(m.state_groups) == 1
    m.allocate_storage("cpu")
    assert m.kv_groups[0].k.shape == (2, 10, 2, 8, 16) and m.kv_groups[0].v.shape == (2, 10, 2, 8, 24)
    assert m.state_groups[0].data.shape == (2, 2, 3, 144)


def test_plain_grouped_norm():
    x = torch.tensor([[3.0, 4.0, 0.1, 0.0, 1.0, 1.0]], dtype=F)
    got = plain.group_norm(x, torch.full((6,), 2.0), 3, 0.5)
    want = [3 / math.sqrt(13.0), 4 / math.sqrt(13.0), 0.1 / math.sqrt(0.505), 0.0, 1 / math.sqrt(1.5), 1 / math.sqrt(1.5)]
    assert torch.allclose(got[0], 2 * torch.tensor(want, dtype=F))
    whole = plain.group_norm(x, torch.ones(6), 1, 0.0)
    assert torch.allclose(whole, x / (x * x).mean().sqrt())


def test_plain_convolution():
    u = torch.tensor([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0], [4.0, 40.0]], dtype=F)
    w = torch.tensor([[100.0, 10.0, 1.0], [0.0, 0.0, 1.0]])
    got = plain.causal_conv(u, w)
    assert got[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0] and got[:, 1].tolist() == [10.0, 20.0, 30.0, 40.0]


def test_plain_frequencies_and_rotation():
    f, mult = plain.frequencies({"base": 100.0, "dims": 8})
    assert f == pytest.approx([1.0, 100 ** -0.25, 0.1, 100 ** -0.75]) and mult == 1.0
    # a ramp by hand: dims 8, base 100, original 64; pair_of(t) = 8 ln(64 / (2 pi t)) / (2 ln 100)
    pair = lambda t: 8 * math.log(64 / (2 * math.pi * t)) / (2 * math.log(100))
    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 0.5}}
    lo, hi = max(math.floor(pair(4.0)), 0), min(math.ceil(pair(0.5)), 7)
    assert lo == 0 and hi == 3
    g, mult = plain.frequencies(rot)
    for i in range(4):
        r = i / 3
        assert g[i] == pytest.approx(f[i] / 4 * r + f[i] * (1 - r))
    assert mult == pytest.approx(0.1 * math.log(4) + 1)
    from inf_engine_b200.config import PositionSpec, YarnScaling
    from inf_engine_b200.parts.positions import partial_rotation_frequencies
    for s in ((4.0, 64.0, 4.0, 0.5), (8.0, 2048.0, 32.0, 1.0), (2.0, 16.0, 3.0, 3.0)):
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), s))
        a, ma = plain.frequencies(rot)
        b, mb = partial_rotation_frequencies(PositionSpec(kind="rotary_partial", theta=100.0, rot_dims=8, yarn=YarnScaling(*s)))
        assert b.tolist() == pytest.approx(a) and mb == pytest.approx(ma)
    x = torch.randn(3, 1, 10, dtype=F)
    y = plain.rotate(x, {"base": 100.0, "dims": 8})
    assert torch.equal(y[:, :, 8:], x[:, :, 8:]) and torch.equal(y[0], x[0])
    z = torch.view_as_complex(x[2, 0, :8].reshape(4, 2).contiguous()) * torch.polar(torch.ones(4, dtype=F), 2 * torch.tensor(f, dtype=F))
    assert torch.allclose(y[2, 0, :8].reshape(4, 2), torch.view_as_real(z))


def test_plain_weights():
    g = torch.Generator().manual_seed(0)
    q, k = 3 * torch.randn(5, 2, 4, generator=g, dtype=F), torch.randn(5, 2, 4, generator=g, dtype=F)
    p = plain.weights(q, k, 0.5, 1.5)
    s = 1.5 * torch.tanh((k[:4, 1] @ q[3, 1]) * 0.5 / 1.5)
    assert torch.allclose(p[1, 3, :4], torch.exp(s) / (1 + torch.exp(s).sum())) and float(p[1, 3, 4]) == 0.0
    s = (k[:1, 0] @ q[0, 0]) * 0.5
    assert torch.allclose(plain.weights(q, k, 0.5, None)[0, 0, :1], torch.sigmoid(s))      # one key and the constant
    assert torch.allclose(plain.weights(q, k, 0.5, None, sink=False).sum(-1), torch.ones(2, 5, dtype=F))


def test_plain_router():
    # the largest score decides a group, not the sum of the two largest
    z = torch.tensor([[2.0, -3.0, 1.9, 1.8, 0.5, 1.0]], dtype=F)
    w = {"router": torch.eye(6)}
    ids, wts = plain.route(z, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}, w, "")
    assert ids == [[0, 1]]
    s = torch.softmax(z[0], -1)
    assert wts[0] == pytest.approx([float(s[0] / (s[0] + s[1])), float(s[1] / (s[0] + s[1]))])
    ids, _ = plain.route(z, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}}, w, "")
    assert ids == [[0, 2, 3]]
    ids, _ = plain.route(z, {"experts": 6, "top": 4}, w, "")
    assert ids == [[0, 2, 3, 5]]


def test_every_mechanism_matters_in_the_test_models(tmp_path):
    """Leaving a mechanism out of the plain model moves its logits: a test model in which it did not would not test it."""
    cfg, w = plain_inputs(make_nurilorn_dir(tmp_path, "nur_a"))
    toks = random_tokens(cfg["vocab"], 60, 9)
    base = plain.forward(cfg, w, toks)

    def moved(change=None, w2=None):
        c = copy.deepcopy(cfg)
        if change is not None:
            change(c)
        other = plain.forward(c, w2 or w, toks)
        return float(((other - base).norm(dim=-1) / base.norm(dim=-1)).max())

    mixer = lambda c, i: c["layers"][i]["mixer"]
    for change in (lambda c: c["norm"].update(groups=1), lambda c: c["embedding"].update(scale=2.5),
                   lambda c: c.update(residual_mult=0.8), lambda c: c.update(logit_scale=0.5),
                   lambda c: mixer(c, 0).update(softcap=None), lambda c: mixer(c, 2).update(softcap=None),
                   lambda c: mixer(c, 0)["rot"].pop("scaling"), lambda c: mixer(c, 3)["rot"].update(dims=6),
                   lambda c: mixer(c, 2)["rot"].update(base=400.0), lambda c: mixer(c, 0).update(v_mix=False),
                   lambda c: c["layers"][0]["mlp"].update(limit=2.0), lambda c: c["layers"][2]["mlp"]["expert"].update(limit=2.0),
                   lambda c: c["layers"][2]["mlp"]["router"]["groups"].update(count=1, keep=1),
                   lambda c: c["layers"][2]["mlp"]["router"].update(top=2)):
        assert moved(change) > 0.003, change
    for name in ("l0.mix.q.conv", "l0.mix.k.conv", "l0.mix.v.conv", "l1.mix.v.conv", "l2.mix.vmix", "l3.mix.vmix", "l0.ls1", "l0.ls2",
                 "l1.ls1", "l2.ls2", "l0.norm1", "l2.norm2", "final.norm", "l0.mix.g", "l2.mlp.router"):
        w2 = dict(w)
        if name.endswith(".conv"):
            w2[name] = torch.zeros_like(w[name])
            w2[name][:, -1] = w[name][:, -1]
        elif name.endswith((".vmix", ".g", ".router")):
            w2[name] = torch.zeros_like(w[name])
        else:
            w2[name] = torch.ones_like(w[name])
        assert moved(w2=w2) > 0.003, name
    w2 = dict(w)
    w2["l0.mix.vmix"] = torch.tensor(0.1)                       # the first mixing layer's own share is idle
    assert moved(w2=w2) == 0.0
    kept = plain.weights
    try:
        plain.weights = lambda q, k, scale, cap, sink=True: kept(q, k, scale, cap, sink=False)
        assert moved() > 0.003
    finally:
        plain.weights = kept
