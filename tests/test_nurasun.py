"""The Nurasun family without a GPU: configuration and its errors, the tensor table, the cache groups its layers ask for,
and the plain implementation's own consistency (dynamic tanh, rotation in halves, chunks, values that are the keys, a
compressed vector read by another layer, the router, the squared relu, gelu), each by hand on small numbers."""

import copy
import math

import pytest
import torch

import plain_nurasun as plain
from nurasun_models import MODELS, make_nurasun_dir, steady_routers
from helpers import plain_inputs, random_tokens

from inf_engine_b200.cache.manager import CacheManager, CacheRequirement
from inf_engine_b200.config import ConfigError, NurasunConfig, parse_config_dict
from inf_engine_b200.parts import expected_tensors

F = torch.float64


def test_config_round_trip_and_specs():
    for name, d in MODELS.items():
        cfg = parse_config_dict(d)
        assert isinstance(cfg, NurasunConfig)
        assert cfg.to_hf_dict() == d, name
        spec = cfg.model_spec()
        assert spec.kind == "decoder" and spec.head == "head" and spec.logit_softcap == d.get("logit_softcap")
        assert spec.final_norm.kind == "tanh_norm" and spec.final_norm.alpha == "final.norm.alpha" and spec.final_norm.bias == "final.norm.b"
        for i, (blk, entry, L) in enumerate(zip(spec.layers, spec.schedule, d["layers"])):
            m, x = L["mixer"], blk.mixer
            assert blk.kind == "parallel" and blk.residual_mult == d["residual_mult"] and blk.ff_norm is None
            assert blk.mixer_norm.alpha == f"l{i}.norm1.alpha" and x.scale == m["scale"]
            assert entry.layer == i and entry.cache_from == m.get("kv_from")
            assert (blk.feedforward is None) == (L["mlp"] is None)
            if L["type"] == "attention":
                assert x.kind == "tied_attention" and x.chunk == m.get("mask", {}).get("size")
                assert (x.n_heads, x.n_kv_heads, x.head_dim) == (m["heads"], m["kv_heads"], m["dim"])
                assert x.position.kind == ("rotary_partial" if "rot" in m else "none")
                if "rot" in m:
                    assert x.position.layout == "halves" and (x.position.theta, x.position.rot_dims) == (m["rot"]["base"], m["rot"]["dims"])
            else:
                assert x.kind == "latent_attention" and x.rot_dim == 0 and x.kv_rank == m["kv_rank"] and x.v_head_dim == m["vdim"]
                assert (x.down_proj == "") == ("kv_from" in m) and x.norm_eps == d["norm"]["eps"]
            if L["mlp"] is not None and L["mlp"]["kind"] == "moe":
                f = blk.feedforward
                assert not f.gated and f.activation == "relu2" and f.score == "sigmoid" and f.shared_gate is None
                assert (f.shared.intermediate if f.shared else None) == L["mlp"].get("shared", {}).get("ff")
            elif L["mlp"] is not None:
                assert blk.feedforward.activation == "gelu_tanh"


def test_what_the_file_may_leave_out():
    d = {"architecture": "Nurasun", "vocab": 50, "width": 24, "norm": {"eps": 1e-5},
         "layers": [{"type": "attention", "mixer": {"heads": 2, "dim": 9, "rot": None, "mask": None}, "mlp": None},
                    {"type": "attention", "mixer": {"heads": 2, "dim": 8, "rot": {"base": 10.0}, "mask": {"size": 7.0}}},
                    {"type": "latent_attention", "mixer": {"heads": 2, "dim": 4, "kv_rank": 6, "kv_from": None},
                     "mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 3, "top": 2}, "shared": None}}]}
    cfg = parse_config_dict(d)
    a, b, c = cfg.layers
    assert cfg.residual_mult == 1.0 and cfg.logit_softcap is None and cfg.model_spec().logit_softcap is None
    assert a.mixer.kv_heads == 2 and a.mixer.scale == pytest.approx(1 / 3) and a.mixer.rot_dims == 0 and a.mixer.chunk is None
    assert b.mixer.rot_dims == 8 and b.mixer.chunk == 7 and b.mlp is None
    assert c.mixer.vdim == 4 and c.mixer.scale == 0.5 and c.mixer.kv_from is None and c.mlp.shared_ff is None


def test_tensor_table():
    t = expected_tensors(parse_config_dict(MODELS["sun_a"]).model_spec())
    assert t["embed"].shape == (211, 60) and t["head"].shape == (211, 60)
    for n in ("l0.norm1", "l0.norm1.b", "l2.norm1", "final.norm", "final.norm.b"):
        assert t[n].shape == (60,), n
    assert t["l0.norm1.alpha"].shape == () and t["final.norm.alpha"].shape == () and "l0.norm2" not in t
    assert t["l0.mix.q"].shape == (64, 60) and t["l0.mix.q.b"].shape == (64,) and t["l0.mix.k.b"].shape == (32,)
    assert "l0.mix.v" not in t and t["l0.mix.o"].shape == (60, 64)
    assert t["l1.mix.dkv"].shape == (22, 60) and t["l1.mix.dkv.norm"].shape == (22,)
    assert t["l1.mix.uk"].shape == (30, 22) and t["l1.mix.uv"].shape == (18, 22) and t["l1.mix.o"].shape == (60, 18)
    assert "l3.mix.dkv" not in t and "l3.mix.dkv.norm" not in t and t["l3.mix.uv"].shape == (70, 22)
    assert t["l1.mlp.router"].shape == (6, 60) and t["l1.mlp.e5.up"].shape == (28, 60) and "l1.mlp.e5.gate" not in t
    assert t["l1.mlp.shared.up"].shape == (20, 60) and t["l1.mlp.shared.down"].shape == (60, 20)
    assert "l2.mlp.up" not in t and t["l3.mlp.gate"].shape == (44, 60)
    assert not any("shared" in n for n in expected_tensors(parse_config_dict(MODELS["sun_b"]).model_spec()) if n.startswith("l1."))


@pytest.mark.parametrize("change, text", [
    (lambda d: d["layers"][0].update(type="mlstm"), "not built"),
    (lambda d: d["layers"][0]["mlp"].update(kind="conv"), "not built"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda d: d["layers"][0]["mixer"].update(vdim=8), "vdim"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].pop("base"), "base"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=7), "cannot be chosen"),
    (lambda d: d["layers"][1]["mlp"]["shared"].update(ff=0), "shared"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=0), "kv_from"),           # no latent layer
    (lambda d: d["layers"][3]["mixer"].update(kv_from=3), "kv_from"),           # itself
    (lambda d: d["layers"][3]["mixer"].update(kv_rank=20), "kv_rank"),
    (lambda d: d["layers"].append(copy.deepcopy(d["layers"][3]) | {"mixer": d["layers"][3]["mixer"] | {"kv_from": 3}}), "kv_from"),
    (lambda d: d.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda d: d.pop("width"), "width"),
    (lambda d: d["norm"].pop("eps"), "eps"),
])
def test_config_errors(change, text):
    d = copy.deepcopy(MODELS["sun_a"])
    change(d)
    with pytest.raises(ConfigError, match=text):
        parse_config_dict(d)


def test_cache_groups_of_the_layers():
    """A layer that reads another's vectors asks for nothing; a layer that rotates nothing keeps one pool; layers with a
    chunk give pages back behind it."""
    tied = lambda g, d, chunk, one: CacheRequirement(kind="kv", n_kv_heads=g, head_dim=d, dtype=torch.float32, chunk=chunk, values_in_keys=one)
    latent = CacheRequirement(kind="kv", n_kv_heads=1, head_dim=22, v_head_dim=22, dtype=torch.float32, values_in_keys=True)
    m = CacheManager([tied(2, 16, 20, False), latent, tied(3, 10, None, True), CacheRequirement(kind="none")], page_size=8,
                     n_pages=10, max_requests=2)
    assert len(m.kv_groups) == 3 and not m.state_groups and m.bindings[3].kind == "none"
    m.allocate_storage("cpu")
    a, b, c = m.kv_groups
    assert a.k.shape == a.v.shape == (1, 10, 2, 8, 16) and a.v is not a.k
    assert b.k.shape == (1, 10, 1, 8, 22) and b.v is b.k and c.k.shape == (1, 10, 3, 8, 10) and c.v is c.k
    assert m.storage_bytes() == 4 * 80 * (2 * 2 * 16 + 22 + 30)
    m.open("r")
    assert m.reserve("r", 50)
    m.advance("r", 50)                       # the next token's chunk starts at 40: five pages lie wholly before it
    assert a.pool.n_held == 2 and b.pool.n_held == c.pool.n_held == 7
    m.check()


def test_a_layer_that_reads_another_must_be_told_where():
    from inf_engine_b200.config import LatentAttentionSpec
    from inf_engine_b200.parts import LatentAttention

    spec = LatentAttentionSpec(kind="latent_attention", hidden=8, n_heads=2, head_dim=4, v_head_dim=4, kv_rank=6, q_proj="q",
                               k_up="uk", v_up="uv", o_proj="o")
    assert set(LatentAttention.expected_tensors(spec)) == {"q", "uk", "uv", "o"}
    part = LatentAttention.__new__(LatentAttention)
    part.spec, part.borrows = spec, True
    with pytest.raises(ValueError, match="cache_from"):
        part.cache_requirement()


def test_plain_dynamic_tanh():
    x = torch.tensor([[0.0, 1.0, -2.0, 40.0]], dtype=F)
    w = {"n": torch.tensor([1.0, 2.0, 0.5, -1.0]), "n.b": torch.tensor([0.25, 0.0, 1.0, 3.0]), "n.alpha": torch.tensor(0.5)}
    want = [0.25, 2 * math.tanh(0.5), 0.5 * math.tanh(-1.0) + 1.0, 2.0]
    assert plain.tanh_norm(x, w, "n")[0].tolist() == pytest.approx(want)


def test_plain_rotation():
    x = torch.randn(4, 2, 10, dtype=F)
    y = plain.rotate(x, {"base": 100.0, "dims": 6})
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.equal(y[0], x[0])
    for i in range(3):
        z = torch.complex(x[3, 1, i], x[3, 1, i + 3]) * torch.polar(torch.tensor(1.0, dtype=F), torch.tensor(3 * 100 ** (-i / 3), dtype=F))
        assert y[3, 1, i].item() == pytest.approx(z.real.item()) and y[3, 1, i + 3].item() == pytest.approx(z.imag.item())
    assert torch.equal(plain.rotate(x, None), x)


def test_plain_chunks():
    q = torch.zeros(7, 1, 2, dtype=F)
    a = plain.weights(q, q, 1.0, 3)[0]
    for i in range(7):
        lo = i // 3 * 3
        assert a[i].tolist() == pytest.approx([1 / (i - lo + 1) if lo <= j <= i else 0.0 for j in range(7)])
    a = plain.weights(q, q, 1.0)[0]
    assert a[6].tolist() == pytest.approx([1 / 7] * 7) and float(a[2, 3]) == 0.0


def test_plain_values_are_the_keys_before_rotation():
    """One key: the output is its projection with the bias, wherever it stands and however it is turned."""
    w = {n: torch.randn(s) for n, s in {"q": (4, 3), "q.b": (4,), "k": (4, 3), "k.b": (4,), "o": (4, 4)}.items()}
    w["o"] = torch.eye(4)
    h = torch.randn(5, 3, dtype=F)
    m = {"heads": 1, "kv_heads": 1, "dim": 4, "scale": 1.0, "rot": {"base": 10.0, "dims": 4}, "mask": {"size": 1}}
    assert torch.allclose(plain.attention(h, m, w, ""), h @ w["k"].to(F).T + w["k.b"].to(F))


def test_plain_latent_layer_that_reads_another():
    h = torch.randn(4, 6, dtype=F)
    w = {n: torch.randn(s) for n, s in {"dkv": (5, 6), "dkv.norm": (5,), "q": (4, 6), "uk": (4, 5), "uv": (6, 5), "o": (6, 6)}.items()}
    c = plain.latent_vector(h, w, "", 0.5)
    z = h @ w["dkv"].to(F).T
    assert torch.allclose(c[2], z[2] / math.sqrt(float((z[2] ** 2).mean()) + 0.5) * w["dkv.norm"].to(F))
    w["o"] = torch.eye(6)
    got = plain.latent_attention(h, c, {"heads": 2, "dim": 2, "vdim": 3, "scale": 0.7}, w, "")
    q, k, v = (h @ w["q"].to(F).T).reshape(4, 2, 2), (c @ w["uk"].to(F).T).reshape(4, 2, 2), (c @ w["uv"].to(F).T).reshape(4, 2, 3)
    p = torch.softmax(k[:3, 1] @ q[2, 1] * 0.7, 0)
    assert torch.allclose(got[2, 3:], p @ v[:3, 1])


def test_plain_router_and_experts():
    z = torch.tensor([[2.0, -3.0, 1.9, 1.8]], dtype=F)
    ids, wts = plain.route(z, {"experts": 4, "top": 2}, {"router": torch.eye(4)}, "")
    s = torch.sigmoid(z[0])
    assert ids == [[0, 2]] and wts[0] == pytest.approx([float(s[0] / (s[0] + s[2])), float(s[2] / (s[0] + s[2]))])
    w = {"up": torch.tensor([[1.0, 0.0], [0.0, 1.0]]), "down": torch.tensor([[1.0, 10.0]])}
    assert plain.squared_relu(torch.tensor([[3.0, -2.0]], dtype=F), w, "").tolist() == [[9.0]]
    assert plain.squared_relu(torch.tensor([[-1.0, 2.0]], dtype=F), w, "").tolist() == [[40.0]]


def test_plain_gelu_and_the_constants_of_the_epilogues():
    x = torch.linspace(-6, 6, 101, dtype=F)
    assert torch.allclose(plain.gelu(x), torch.nn.functional.gelu(x, approximate="tanh"))
    from inf_engine_b200 import kernels
    alpha, limit, offset, cubic = kernels.glu_constants("gelu_tanh")
    assert torch.allclose(x * torch.sigmoid(alpha * x + cubic * x ** 3), plain.gelu(x)) and limit == float("inf") and offset == 0.0
    assert kernels.glu_constants("silu") == (1.0, float("inf"), 0.0, 0.0)
    with pytest.raises(KeyError):
        kernels.glu_constants("softplus")


def test_every_mechanism_matters_in_the_test_models(tmp_path):
    """Leaving a mechanism out of the plain model moves its logits: a test model in which it did not would not test it."""
    cfg, w = plain_inputs(make_nurasun_dir(tmp_path, "sun_a"))
    toks = random_tokens(cfg["vocab"], 60, 9)
    base = plain.forward(cfg, w, toks)

    def moved(change=None, w2=None):
        c = copy.deepcopy(cfg)
        if change is not None:
            change(c)
        other = plain.forward(c, w2 or w, toks)
        return float(((other - base).norm(dim=-1) / base.norm(dim=-1)).max())

    mixer = lambda c, i: c["layers"][i]["mixer"]
    for change in (lambda c: c["norm"].update(eps=0.3), lambda c: c.update(residual_mult=0.75), lambda c: c.update(logit_softcap=3.0),
                   lambda c: c.pop("logit_softcap"), lambda c: mixer(c, 0)["mask"].update(size=21), lambda c: mixer(c, 0).pop("mask"),
                   lambda c: mixer(c, 0)["rot"].update(dims=6), lambda c: mixer(c, 0)["rot"].update(base=400.0),
                   lambda c: mixer(c, 0).pop("rot"), lambda c: mixer(c, 1).update(scale=0.4), lambda c: mixer(c, 3).update(scale=0.4),
                   lambda c: mixer(c, 2).update(mask={"size": 30}), lambda c: mixer(c, 2).update(rot={"base": 50.0, "dims": 10}),
                   lambda c: c["layers"][1]["mlp"].pop("shared"), lambda c: c["layers"][1]["mlp"]["router"].update(top=2)):
        assert moved(change) > 0.003, change
    for name in ("l0.norm1.alpha", "l1.norm1.b", "l2.norm1", "final.norm.alpha", "final.norm.b", "l0.mix.q.b", "l0.mix.k.b",
                 "l2.mix.k.b", "l1.mix.dkv.norm", "l1.mlp.router", "l3.mix.uk"):
        w2 = dict(w)
        w2[name] = torch.zeros_like(w[name]) if not name.endswith((".alpha", ".norm", ".norm1")) else torch.ones_like(w[name])
        assert moved(w2=w2) > 0.003, name
    # values turned with the keys would be another model
    kept = plain.rotate
    calls = []
    try:
        def turned(x, rot):
            calls.append(1)
            y = kept(x, rot)
            if rot and len(calls) % 2 == 0:
                x.copy_(y)                   # the keys' tensor is the values' too
            return y
        plain.rotate = turned
        assert moved() > 0.003
    finally:
        plain.rotate = kept
    # a reader with vectors of its own (another gain than the read layer's) would be another model
    latent = plain.latent_vector
    try:
        plain.latent_vector = lambda *a, **k: torch.flip(latent(*a, **k), dims=[-1])
        assert moved() > 0.003
    finally:
        plain.latent_vector = latent


def test_steady_routers_decide_by_a_wide_margin(tmp_path):
    for name in ("sun_a", "sun_b", "sun_c", "sun_w", "sun_t", "sun_moe"):
        cfg, w = plain_inputs(make_nurasun_dir(tmp_path, name, fix=steady_routers))
        gaps = []
        plain.forward(cfg, w, random_tokens(cfg["vocab"], 40, 3), gaps=gaps)
        assert min(float(g.min()) for g in gaps) > 0.1, name
