"""Typed configuration of the Nurasun decoder, read from ``config.json``.

A Nurasun model runs layers whose two sublayers read the output of one norm side by side, ``x += c * (mixer(h) + ff(h))``
with h = norm(x) and one constant c for the whole model.  The norm is a dynamic tanh, ``tanh(alpha x) * gain + offset``
with one learned alpha; the same kind of norm stands before an untied head, whose logits are capped by a hyperbolic
tangent.  Two kinds of layer, in whatever order the file lists them:

* ``attention``: grouped-query attention without a value projection (the values are the projected keys before their
  rotation), biases on queries and keys, the first dimensions of every head turned in halves, an optional mask that keeps
  a query inside its chunk of positions.
* ``latent_attention``: causal attention without positions whose keys and values are expanded from one RMS-normed
  compressed vector a token; a layer with ``kv_from`` compresses nothing and reads the vectors of the layer it names.

The feed-forward is dense (gate and up, the tanh form of gelu) or a mixture of experts without a gate (up, the square of
relu) chosen by sigmoid scores, with a shared expert of the same form that every token runs.

    {"architecture": "Nurasun", "vocab": V, "width": d, "norm": {"eps": e}, "residual_mult": c, "logit_softcap": t,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "rot": {"base", "dims"}, "mask": {"size"}}, "mlp": M | null},
                {"type": "latent_attention", "mixer": {"heads", "dim", "vdim", "kv_rank", "scale", "kv_from"}, "mlp": M | null}]}
    M = {"kind": "dense", "ff": f}
      | {"kind": "moe", "expert": {"ff": f}, "router": {"experts": E, "top": k}, "shared": {"ff": s}}

Tensor names: ``embed``, ``l<i>.norm1`` (+ ``.alpha``, ``.b``), ``l<i>.mix.q|k`` (+ ``.b``), ``l<i>.mix.o``,
``l<i>.mix.dkv`` (+ ``.norm``), ``l<i>.mix.uk|uv``, ``l<i>.mlp.gate|up|down``, ``l<i>.mlp.router``,
``l<i>.mlp.e<j>.up|down``, ``l<i>.mlp.shared.up|down``, ``final.norm`` (+ ``.alpha``, ``.b``), ``head``.
"""

from __future__ import annotations

from dataclasses import dataclass, field

from .fovunex import NO_POSITION_LIMIT, _need, _nonneg_int, _pos_int
from .llama import ConfigError
from .nurilorn import _positive
from .spec import (
    BlockSpec,
    GatedMLPSpec,
    LatentAttentionSpec,
    MLPSpec,
    ModelSpec,
    NormSpec,
    PositionSpec,
    RoutedExpertsSpec,
    ScheduleEntry,
    TiedAttentionSpec,
)

# The design fixes this.
ROUTE_WEIGHT_EPS = 1e-20        # added to the sum that the chosen experts' scores are divided by


@dataclass(frozen=True)
class NurasunDense:
    ff: int


@dataclass(frozen=True)
class NurasunMoE:
    ff: int
    experts: int
    top: int
    shared_ff: int | None = None


@dataclass(frozen=True)
class NurasunAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot_base: float = 0.0
    rot_dims: int = 0                           # 0: nothing is turned
    chunk: int | None = None                    # None: every earlier key


@dataclass(frozen=True)
class NurasunLatent:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    kv_from: int | None = None                  # the layer whose compressed vectors are read; None: this layer's own


@dataclass(frozen=True)
class NurasunLayer:
    type: str                                   # "attention" | "latent_attention"
    mixer: NurasunAttention | NurasunLatent
    mlp: NurasunDense | NurasunMoE | None = None


def _parse_attention(m, where: str) -> NurasunAttention:
    heads = _pos_int(_need(m, "heads", where), where + ".heads")
    kv = _pos_int(m.get("kv_heads", heads), where + ".kv_heads")
    if heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} heads are not a multiple of {kv} kv_heads")
    dim = _pos_int(_need(m, "dim", where), where + ".dim")
    vdim = _pos_int(m.get("vdim", dim), where + ".vdim")
    if vdim != dim:
        raise ConfigError(f"config.json: {where}: the values are the keys, so vdim must equal dim={dim}, got {vdim}")
    rot = m.get("rot") or {}
    dims = _nonneg_int(rot.get("dims", dim), where + ".rot.dims") if rot else 0
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim={dim}, got {dims}")
    base = _positive(_need(rot, "base", where + ".rot"), where + ".rot.base") if dims else 0.0
    mask = m.get("mask")
    chunk = _pos_int(_need(mask, "size", where + ".mask"), where + ".mask.size") if mask else None
    return NurasunAttention(heads, kv, dim, float(m.get("scale", dim ** -0.5)), base, dims, chunk)


def _parse_latent(m, where: str) -> NurasunLatent:
    dim = _pos_int(_need(m, "dim", where), where + ".dim")
    src = m.get("kv_from")
    return NurasunLatent(_pos_int(_need(m, "heads", where), where + ".heads"), dim,
                         _pos_int(m.get("vdim", dim), where + ".vdim"), _pos_int(_need(m, "kv_rank", where), where + ".kv_rank"),
                         float(m.get("scale", dim ** -0.5)), None if src is None else _nonneg_int(src, where + ".kv_from"))


def _parse_mlp(mlp, where: str):
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind == "dense":
        return NurasunDense(_pos_int(_need(mlp, "ff", where), where + ".ff"))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not built (known: dense, moe)")
    ew, rw, sw = where + ".expert", where + ".router", where + ".shared"
    e, r, shared = _need(mlp, "expert", where), _need(mlp, "router", where), mlp.get("shared")
    experts = _pos_int(_need(r, "experts", rw), rw + ".experts")
    top = _pos_int(_need(r, "top", rw), rw + ".top")
    if top > experts:
        raise ConfigError(f"config.json: {where}: {top} experts cannot be chosen from {experts}")
    return NurasunMoE(_pos_int(_need(e, "ff", ew), ew + ".ff"), experts, top,
                      _pos_int(_need(shared, "ff", sw), sw + ".ff") if shared else None)


@dataclass(frozen=True)
class NurasunConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float = 1.0
    logit_softcap: float | None = None
    layers: tuple[NurasunLayer, ...] = field(default_factory=tuple)
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
    def from_dict(cls, d: dict) -> "NurasunConfig":
        vocab = _pos_int(_need(d, "vocab", "the top level"), "vocab")
        width = _pos_int(_need(d, "width", "the top level"), "width")
        eps = _positive(_need(_need(d, "norm", "the top level"), "eps", "'norm'"), "norm.eps")
        raw = _need(d, "layers", "the top level")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: list[NurasunLayer] = []
        for i, e in enumerate(raw):
            where = f"layers[{i}]"
            kind, m = _need(e, "type", where), _need(e, "mixer", where)
            if kind == "attention":
                mixer = _parse_attention(m, where + ".mixer")
            elif kind == "latent_attention":
                mixer = _parse_latent(m, where + ".mixer")
                j = mixer.kv_from
                if j is not None:
                    src = layers[j].mixer if j < i and layers[j].type == kind else None
                    if src is None or src.kv_from is not None:
                        raise ConfigError(f"config.json: {where}.mixer.kv_from must name an earlier latent_attention layer "
                                          f"with a compressed vector of its own, got {j}")
                    if src.kv_rank != mixer.kv_rank:
                        raise ConfigError(f"config.json: {where}.mixer.kv_rank is {mixer.kv_rank}, that of the layer it reads "
                                          f"({j}) is {src.kv_rank}")
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not built (known: attention, latent_attention)")
            layers.append(NurasunLayer(kind, mixer, _parse_mlp(e.get("mlp"), where + ".mlp")))
        cap = d.get("logit_softcap")
        return cls(architecture=str(d.get("architecture") or (d.get("architectures") or ["Nurasun"])[0]), vocab=vocab,
                   width=width, norm_eps=eps, residual_mult=float(d.get("residual_mult", 1.0)),
                   logit_softcap=_positive(cap, "logit_softcap") if cap else None, layers=tuple(layers),
                   eos_token_id=d.get("eos_token_id"))

    def to_hf_dict(self) -> dict:
        layers = []
        for L in self.layers:
            x, f = L.mixer, L.mlp
            if L.type == "attention":
                mixer = {"heads": x.heads, "kv_heads": x.kv_heads, "dim": x.dim, "vdim": x.dim, "scale": x.scale}
                if x.rot_dims:
                    mixer["rot"] = {"base": x.rot_base, "dims": x.rot_dims}
                if x.chunk is not None:
                    mixer["mask"] = {"size": x.chunk}
            else:
                mixer = {"heads": x.heads, "dim": x.dim, "vdim": x.vdim, "kv_rank": x.kv_rank, "scale": x.scale}
                if x.kv_from is not None:
                    mixer["kv_from"] = x.kv_from
            if f is None:
                mlp = None
            elif isinstance(f, NurasunDense):
                mlp = {"kind": "dense", "ff": f.ff}
            else:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff is not None:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"type": L.type, "mixer": mixer, "mlp": mlp})
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "residual_mult": self.residual_mult, "layers": layers}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.eos_token_id is not None:
            out["eos_token_id"] = self.eos_token_id
        return out

    to_dict = to_hf_dict

    # ---- the model as data
    def _norm(self, name: str) -> NormSpec:
        return NormSpec("tanh_norm", self.width, self.norm_eps, name, bias=name + ".b", alpha=name + ".alpha")

    def _mixer_spec(self, L: NurasunLayer, m: str):
        x = L.mixer
        if L.type == "attention":
            position = PositionSpec(kind="none")
            if x.rot_dims:
                position = PositionSpec(kind="rotary_partial", head_dim=x.dim, theta=x.rot_base, rot_dims=x.rot_dims,
                                        layout="halves")
            return TiedAttentionSpec(kind="tied_attention", hidden=self.width, n_heads=x.heads, n_kv_heads=x.kv_heads,
                                     head_dim=x.dim, scale=x.scale, position=position, chunk=x.chunk, q_proj=m + "q",
                                     k_proj=m + "k", q_bias=m + "q.b", k_bias=m + "k.b", o_proj=m + "o")
        own = x.kv_from is None
        return LatentAttentionSpec(
            kind="latent_attention", hidden=self.width, n_heads=x.heads, head_dim=x.dim, rot_dim=0, v_head_dim=x.vdim,
            kv_rank=x.kv_rank, scale=x.scale, norm_eps=self.norm_eps, q_proj=m + "q", down_proj=m + "dkv" if own else "",
            latent_norm=m + "dkv.norm" if own else "", k_up=m + "uk", v_up=m + "uv", o_proj=m + "o")

    def _ff_spec(self, x, f: str):
        if x is None:
            return None
        if isinstance(x, NurasunDense):
            return GatedMLPSpec(kind="gated_mlp", hidden=self.width, intermediate=x.ff, activation="gelu_tanh",
                                gate_proj=f + "gate", up_proj=f + "up", down_proj=f + "down")
        shared = None
        if x.shared_ff is not None:
            shared = MLPSpec(kind="mlp", hidden=self.width, intermediate=x.shared_ff, activation="relu2",
                             up_proj=f + "shared.up", down_proj=f + "shared.down")
        return RoutedExpertsSpec(kind="routed_experts", hidden=self.width, intermediate=x.ff, n_experts=x.experts, top=x.top,
                                 weight_eps=ROUTE_WEIGHT_EPS, router=f + "router", expert_prefix=f + "e", shared=shared,
                                 score="sigmoid", gated=False, activation="relu2")

    def model_spec(self) -> ModelSpec:
        layers = tuple(BlockSpec(kind="parallel", mixer_norm=self._norm(f"l{i}.norm1"), mixer=self._mixer_spec(L, f"l{i}.mix."),
                                 ff_norm=None, feedforward=self._ff_spec(L.mlp, f"l{i}.mlp."), residual_mult=self.residual_mult)
                       for i, L in enumerate(self.layers))
        # a run whose mixer reads another layer's compressed vectors reads that run's cache
        schedule = tuple(ScheduleEntry(layer=i, cache_from=getattr(L.mixer, "kv_from", None)) for i, L in enumerate(self.layers))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden=self.width, max_positions=NO_POSITION_LIMIT,
            embedding="embed", layers=layers, schedule=schedule, final_norm=self._norm("final.norm"), head="head",
            logit_softcap=self.logit_softcap)
