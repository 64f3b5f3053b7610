"""Typed configuration of the Nurilorn decoder, read from ``config.json``.

A Nurilorn model multiplies its token embedding by a constant and runs pre-norm layers, ``x += c * ls1 * mixer(norm1(x))``
and ``x += c * ls2 * ff(norm2(x))``, with one constant c for the whole model, a learned number per coordinate for each
sublayer, and an RMS norm that norms each of several equal parts of the row by itself.  It ends in the same kind of norm
and an untied head whose logits are multiplied by a constant.  One kind of mixer:

* ``attention``: causal grouped-query attention; q, k and v each pass a short causal convolution over time; the first
  dimensions of every query and key head are turned in neighbouring pairs, optionally with frequencies blended for a
  longer context (YaRN); scores are capped by a hyperbolic tangent; the softmax's denominator holds one more term, 1;
  layers that say so blend their values with those of the first such layer (same token); every head's output passes a
  sigmoid gate.

The feed-forward is dense or a mixture of experts, both with clamped gate and up branches and the activation
``g sigmoid(1.702 g) (u + 1)``; the router's scores are a softmax over all experts, the best groups of neighbouring
experts (by their largest score) are kept, and the chosen scores are divided by their sum.

    {"architecture": "Nurilorn", "vocab": V, "width": d, "norm": {"eps": e, "groups": g}, "embedding": {"scale": s},
     "residual_mult": c, "logit_scale": t,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "conv", "scale", "softcap", "v_mix",
                           "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}}, "mlp": M | null}]}
    M = {"kind": "dense", "ff": f, "limit": l}
      | {"kind": "moe", "expert": {"ff": f, "limit": l}, "router": {"experts": E, "top": k, "groups": {"count", "keep"}}}

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.ls1``, ``l<i>.ls2``, ``l<i>.mix.q|k|v`` (+ ``.conv``),
``l<i>.mix.vmix|g|o``, ``l<i>.mlp.gate|up|down``, ``l<i>.mlp.router``, ``l<i>.mlp.e<j>.gate|up|down``, ``final.norm``,
``head``.
"""

from __future__ import annotations

from dataclasses import dataclass, field

from .fovunex import NO_POSITION_LIMIT, _need, _nonneg_int, _pos_int
from .llama import ConfigError
from .spec import (
    BlockSpec,
    ConvAttentionSpec,
    GatedMLPSpec,
    ModelSpec,
    NormSpec,
    PositionSpec,
    RoutedExpertsSpec,
    ScheduleEntry,
    ShortConvSpec,
    YarnScaling,
)

# The design fixes these.
ACT_ALPHA = 1.702               # the activation is g sigmoid(1.702 g) (u + 1)
UP_OFFSET = 1.0
SINK_LOGIT = 0.0                # the softmax's denominator also holds exp(0)
ROUTE_WEIGHT_EPS = 1e-20        # added to the sum that the chosen experts' scores are divided by
YARN_MULT_SLOPE = 0.1           # cosine and sine times 0.1 ln(factor) + 1


@dataclass(frozen=True)
class NurilornDense:
    ff: int
    limit: float


@dataclass(frozen=True)
class NurilornMoE:
    ff: int
    limit: float
    experts: int
    top: int
    groups: int = 1
    keep_groups: int = 1


@dataclass(frozen=True)
class NurilornRotation:
    base: float
    dims: int
    yarn: YarnScaling | None = None


@dataclass(frozen=True)
class NurilornAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int = 0                               # taps; 0: no convolutions
    softcap: float | None = None
    v_mix: bool = False
    rot: NurilornRotation | None = None


@dataclass(frozen=True)
class NurilornLayer:
    type: str                                   # "attention"
    mixer: NurilornAttention
    mlp: NurilornDense | NurilornMoE | None = None


def _positive(v, what: str) -> float:
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not v > 0:
        raise ConfigError(f"config.json: {what} must be positive, got {v!r}")
    return float(v)


def _parse_rot(rot, dim: int, where: str) -> NurilornRotation | None:
    if not rot:
        return None
    dims = _nonneg_int(rot.get("dims", dim), where + ".dims")
    if dims == 0:
        return None
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where}.dims must be even and at most dim={dim}, got {dims}")
    base = _positive(_need(rot, "base", where), where + ".base")
    s = rot.get("scaling")
    if not s:
        return NurilornRotation(base, dims)
    sw = where + ".scaling"
    if base == 1.0:
        raise ConfigError(f"config.json: {sw} needs a base other than 1")
    yarn = YarnScaling(**{key: _positive(_need(s, key, sw), f"{sw}.{key}") for key in ("factor", "original", "fast", "slow")},
                       mult_slope=YARN_MULT_SLOPE)
    return NurilornRotation(base, dims, yarn)


def _parse_attention(m, where: str) -> NurilornAttention:
    heads = _pos_int(_need(m, "heads", where), where + ".heads")
    kv = _pos_int(m.get("kv_heads", heads), where + ".kv_heads")
    if heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} heads are not a multiple of {kv} kv_heads")
    dim = _pos_int(_need(m, "dim", where), where + ".dim")
    vdim = _pos_int(m.get("vdim", dim), where + ".vdim")
    cap = m.get("softcap")
    return NurilornAttention(heads, kv, dim, vdim, float(m.get("scale", dim ** -0.5)),
                             _nonneg_int(m.get("conv") or 0, where + ".conv"),
                             _positive(cap, where + ".softcap") if cap else None, bool(m.get("v_mix", False)),
                             _parse_rot(m.get("rot"), dim, where + ".rot"))


def _parse_mlp(mlp, where: str):
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind == "dense":
        return NurilornDense(_pos_int(_need(mlp, "ff", where), where + ".ff"),
                             _positive(_need(mlp, "limit", where), where + ".limit"))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not built (known: dense, moe)")
    ew, rw = where + ".expert", where + ".router"
    e, r = _need(mlp, "expert", where), _need(mlp, "router", where)
    experts = _pos_int(_need(r, "experts", rw), rw + ".experts")
    top = _pos_int(_need(r, "top", rw), rw + ".top")
    g = r.get("groups") or {}
    groups = _pos_int(g.get("count", 1), rw + ".groups.count")
    keep = _pos_int(g.get("keep", groups), rw + ".groups.keep")
    if experts % groups:
        raise ConfigError(f"config.json: {where}: {experts} experts do not form {groups} equal groups")
    if keep > groups:
        raise ConfigError(f"config.json: {where}: {keep} groups cannot be kept out of {groups}")
    if top > keep * (experts // groups):
        raise ConfigError(f"config.json: {where}: {top} experts cannot be chosen from {keep} groups of {experts // groups}")
    return NurilornMoE(_pos_int(_need(e, "ff", ew), ew + ".ff"), _positive(_need(e, "limit", ew), ew + ".limit"), experts,
                       top, groups, keep)


@dataclass(frozen=True)
class NurilornConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int = 1
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    layers: tuple[NurilornLayer, ...] = field(default_factory=tuple)
    eos_token_id: int | None = None

    # names other parts of the package ask a configuration for
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        return NO_POSITION_LIMIT

    # ---- reading and writing config.json
    @classmethod
    def from_dict(cls, d: dict) -> "NurilornConfig":
        vocab = _pos_int(_need(d, "vocab", "the top level"), "vocab")
        width = _pos_int(_need(d, "width", "the top level"), "width")
        norm = _need(d, "norm", "the top level")
        eps = _positive(_need(norm, "eps", "'norm'"), "norm.eps")
        groups = _pos_int(norm.get("groups", 1), "norm.groups")
        if width % groups:
            raise ConfigError(f"config.json: a width of {width} does not split into {groups} equal norm groups")
        raw = _need(d, "layers", "the top level")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(raw):
            where = f"layers[{i}]"
            kind = _need(e, "type", where)
            if kind != "attention":
                raise ConfigError(f"config.json: {where}.type {kind!r} is not built (known: attention)")
            layers.append(NurilornLayer(kind, _parse_attention(_need(e, "mixer", where), where + ".mixer"),
                                        _parse_mlp(e.get("mlp"), where + ".mlp")))
        mixing = [(i, L.mixer.kv_heads * L.mixer.vdim) for i, L in enumerate(layers) if L.mixer.v_mix]
        for i, size in mixing:
            if size != mixing[0][1]:
                raise ConfigError(f"config.json: layers[{i}] mixes {size} values a token, layers[{mixing[0][0]}] has {mixing[0][1]}")
        return cls(architecture=str(d.get("architecture") or (d.get("architectures") or ["Nurilorn"])[0]), vocab=vocab,
                   width=width, norm_eps=eps, norm_groups=groups,
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   residual_mult=float(d.get("residual_mult", 1.0)), logit_scale=float(d.get("logit_scale", 1.0)),
                   layers=tuple(layers), eos_token_id=d.get("eos_token_id"))

    def to_hf_dict(self) -> dict:
        layers = []
        for L in self.layers:
            x = L.mixer
            mixer = {"heads": x.heads, "kv_heads": x.kv_heads, "dim": x.dim, "vdim": x.vdim, "scale": x.scale,
                     "v_mix": x.v_mix}
            if x.conv:
                mixer["conv"] = x.conv
            if x.softcap is not None:
                mixer["softcap"] = x.softcap
            if x.rot is not None:
                rot = {"base": x.rot.base, "dims": x.rot.dims}
                y = x.rot.yarn
                if y is not None:
                    rot["scaling"] = {"factor": y.factor, "original": y.original, "fast": y.fast, "slow": y.slow}
                mixer["rot"] = rot
            f = L.mlp
            if f is None:
                mlp = None
            elif isinstance(f, NurilornDense):
                mlp = {"kind": "dense", "ff": f.ff, "limit": f.limit}
            else:
                mlp = {"kind": "moe", "expert": {"ff": f.ff, "limit": f.limit},
                       "router": {"experts": f.experts, "top": f.top, "groups": {"count": f.groups, "keep": f.keep_groups}}}
            layers.append({"type": L.type, "mixer": mixer, "mlp": mlp})
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "embedding": {"scale": self.embedding_scale},
               "residual_mult": self.residual_mult, "logit_scale": self.logit_scale, "layers": layers}
        if self.eos_token_id is not None:
            out["eos_token_id"] = self.eos_token_id
        return out

    to_dict = to_hf_dict

    # ---- the model as data
    def _norm(self, name: str, out_scale: float = 1.0) -> NormSpec:
        return NormSpec("grouped_rmsnorm", self.width, self.norm_eps, name, groups=self.norm_groups, out_scale=out_scale)

    def _mixer_spec(self, x: NurilornAttention, m: str, first_mixing: bool) -> ConvAttentionSpec:
        position = PositionSpec(kind="none")
        if x.rot is not None:
            position = PositionSpec(kind="rotary_partial", head_dim=x.dim, theta=x.rot.base, rot_dims=x.rot.dims,
                                    layout="neighbours", yarn=x.rot.yarn)
        conv = lambda name: ShortConvSpec(x.conv, m + name + ".conv") if x.conv else None
        return ConvAttentionSpec(
            kind="conv_attention", hidden=self.width, n_heads=x.heads, n_kv_heads=x.kv_heads, head_dim=x.dim,
            v_head_dim=x.vdim, scale=x.scale, softcap=x.softcap, sink=SINK_LOGIT, position=position, q_proj=m + "q",
            k_proj=m + "k", v_proj=m + "v", q_conv=conv("q"), k_conv=conv("k"), v_conv=conv("v"),
            v_keep=x.v_mix and first_mixing, v_mix=m + "vmix" if x.v_mix and not first_mixing else None,
            head_gate=m + "g", o_proj=m + "o")

    def _ff_spec(self, x, f: str):
        act = dict(activation="clamped_swish", act_alpha=ACT_ALPHA, act_limit=x.limit, up_offset=UP_OFFSET)
        if isinstance(x, NurilornDense):
            return GatedMLPSpec(kind="gated_mlp", hidden=self.width, intermediate=x.ff, gate_proj=f + "gate",
                                up_proj=f + "up", down_proj=f + "down", **act)
        return RoutedExpertsSpec(kind="routed_experts", hidden=self.width, intermediate=x.ff, n_experts=x.experts, top=x.top,
                                 n_groups=x.groups, keep_groups=x.keep_groups, weight_eps=ROUTE_WEIGHT_EPS,
                                 router=f + "router", expert_prefix=f + "e", score="softmax", group_score="max", **act)

    def model_spec(self) -> ModelSpec:
        layers, optional = [], []
        mixing = [i for i, L in enumerate(self.layers) if L.mixer.v_mix]
        for i, L in enumerate(self.layers):
            p = f"l{i}."
            first = bool(mixing) and i == mixing[0]
            if first or not L.mixer.v_mix:
                optional.append(p + "mix.vmix")              # nothing is mixed in: the tensor, if there is one, is idle
            ff_norm, ff = None, None
            if L.mlp is not None:
                ff_norm, ff = self._norm(p + "norm2"), self._ff_spec(L.mlp, p + "mlp.")
            else:
                optional += [p + "norm2", p + "ls2"]         # a layer without a feed-forward has no use for them
            layers.append(BlockSpec(kind="scaled_prenorm", mixer_norm=self._norm(p + "norm1"),
                                    mixer=self._mixer_spec(L.mixer, p + "mix.", first), ff_norm=ff_norm, feedforward=ff,
                                    residual_mult=self.residual_mult, mixer_scale=p + "ls1", ff_scale=p + "ls2"))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden=self.width, max_positions=NO_POSITION_LIMIT,
            embedding="embed", layers=tuple(layers), schedule=tuple(ScheduleEntry(layer=i) for i in range(len(layers))),
            final_norm=self._norm("final.norm", self.logit_scale), head="head", embedding_scale=self.embedding_scale,
            optional_tensors=tuple(optional))
