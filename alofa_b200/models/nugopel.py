"""Nugopel: a decoder with a norm before and after each sublayer whose layers,
listed one by one in config.json, have one of two mixers and optionally a
mixture of experts:

* ``latent_attention``: attention without positions over a cached latent.
  Queries come straight from the input; the score's softmax is the ordinary one
  over every key up to the query; the concatenated heads are gated channel by
  channel.  A layer with ``kv_from`` has no latent of its own: it attends to
  the rows that the named earlier layer caches;
* ``attention``: queries and keys RMS normed over the whole projection, then
  rotated (halves; frequencies scaled by wavelength), a sliding window, one
  added to the softmax's denominator.

The experts are ``Wdown relu(Wup .)^2``; a token takes the ones with the
largest router logits, weighted by the softmax over the chosen logits, plus a
shared one.  The norms around the sublayers and the last one store their
weights less one.  This file only reads the architecture's config keys and
describes the model as a :class:`~alofa_b200.config.spec.ModelSpec`; the parts
it names live in :mod:`alofa_b200.parts` and know nothing about Nugopel.

config.json keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``,
``layers[i].type``, ``layers[i].mixer`` (latent_attention: ``heads, dim, vdim,
kv_rank, scale, kv_from``; attention: ``heads, kv_heads, dim, vdim, scale,
mask.size, rot.{base, dims, scaling.{factor, low, high, original}}``) and
``layers[i].mlp`` (null or ``{kind: moe, expert.ff, router.{experts, top},
shared.ff}``).  Absent ``kv_from``: a latent of its own; absent ``mask``: every
key; absent ``scaling``: frequencies as they are; absent ``shared``: no shared
expert.  Tensor names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b``,
``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

from ..config.json_reader import Keys
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..errors import AlofaError

NAME = "Nugopel"
MAX_POSITION = 1 << 24  # positions are fp32 in the kernels that rotate: whole numbers are exact up to here
SINK = 0.0  # the score of the term that the softmax of "attention" has beside the keys': exp(0), one


@dataclass
class LatentConfig:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    kv_from: Optional[int] = None


@dataclass
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int
    rot_scaling: Optional[dict] = None  # factor, low, high, original
    window: Optional[int] = None


@dataclass
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int = 0  # 0: no shared expert


@dataclass
class NugopelLayer:
    type: str
    mixer: object
    mlp: Optional[ExpertsConfig]


@dataclass
class NugopelConfig:
    vocab: int
    width: int
    eps: float
    layers: list = field(default_factory=list)

    def validate(self, origin: str = "") -> None:
        def need(ok, what, detail):
            if not ok:
                raise AlofaError("parse", what, f"{detail} config={origin}")

        need(self.vocab > 0 and self.width > 0, "vocab and width must be positive", f"vocab={self.vocab} width={self.width}")
        need(self.eps > 0, "norm.eps must be positive", f"eps={self.eps}")
        need(len(self.layers) > 0, "layers must not be empty", "layers=[]")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            where = f"layers[{i}].mixer={m}"
            need(min(m.heads, m.dim, m.vdim) > 0, "mixer sizes must be positive", where)
            if layer.type == "latent_attention":
                need(m.kv_rank > 0, "kv_rank must be positive", where)
                if m.kv_from is not None:
                    need(0 <= m.kv_from < i, "kv_from must name an earlier layer", where)
                    other = self.layers[m.kv_from]
                    need(other.type == "latent_attention" and other.mixer.kv_from is None, "kv_from must name a layer with a latent of its own", where)
                    need(other.mixer.kv_rank == m.kv_rank, "kv_from must name a layer of the same kv_rank", where)
            else:
                need(m.kv_heads > 0 and m.heads % m.kv_heads == 0, "kv_heads must divide heads", where)
                need(m.window is None or m.window > 0, "mask.size must be positive", where)
                need(0 <= m.rot_dims <= m.dim and m.rot_dims % 2 == 0, "rot.dims must be even and at most dim", where)
                need(m.rot_base > 0, "rot.base must be positive", where)
                sc = m.rot_scaling
                need(sc is None or (min(sc.values()) > 0 and sc["high"] >= sc["low"]), "rot.scaling wants positive numbers, high not below low", where)
            f = layer.mlp
            if f is not None:
                where = f"layers[{i}].mlp={f}"
                need(f.ff > 0 and f.shared_ff >= 0, "the experts' inner sizes must be positive", where)
                need(0 < f.top <= f.experts, "router.top must lie in [1, experts]", where)


def _object(obj: dict, key: str, origin: str) -> dict:
    value = obj.get(key)
    if not isinstance(value, dict):
        raise AlofaError("parse", "config key must be an object", f"key={key} config={origin}")
    return value


def _read_mixer(kind: str, obj: dict, origin: str):
    k = Keys(obj, origin)
    if kind == "latent_attention":
        return LatentConfig(k.integer("heads"), k.integer("dim"), k.integer("vdim"), k.integer("kv_rank"), k.number("scale"),
                            k.integer("kv_from") if k.has("kv_from") else None)
    if kind == "attention":
        ro = _object(obj, "rot", origin)
        rot, scaling = Keys(ro, origin), None
        if ro.get("scaling") is not None:
            sk = Keys(_object(ro, "scaling", origin), origin)
            scaling = {n: sk.number(n) for n in ("factor", "low", "high", "original")}
        window = Keys(_object(obj, "mask", origin), origin).integer("size") if obj.get("mask") is not None else None
        return AttentionConfig(k.integer("heads"), k.integer("kv_heads"), k.integer("dim"), k.integer("vdim"), k.number("scale"), rot.number("base"), rot.integer("dims"),
                               scaling, window)
    raise AlofaError("parse", "unknown layer type", f"type={kind} config={origin}")


def _read_mlp(obj, origin: str) -> Optional[ExpertsConfig]:
    if obj is None:
        return None
    if not isinstance(obj, dict):
        raise AlofaError("parse", "mlp must be an object or null", f"config={origin}")
    kind = Keys(obj, origin).string("kind")
    if kind != "moe":
        raise AlofaError("parse", "unknown mlp kind", f"kind={kind} config={origin}")
    r, e = Keys(_object(obj, "router", origin), origin), Keys(_object(obj, "expert", origin), origin)
    shared = 0
    if obj.get("shared") is not None:
        shared = Keys(_object(obj, "shared", origin), origin).integer("ff")
        if shared <= 0:
            raise AlofaError("parse", "shared.ff must be positive", f"ff={shared} config={origin}")
    return ExpertsConfig(r.integer("experts"), r.integer("top"), e.integer("ff"), shared)


def read_config(obj: dict, origin: str) -> NugopelConfig:
    k = Keys(obj, origin)
    layers = obj.get("layers")
    if not isinstance(layers, list):
        raise AlofaError("parse", "config key must be a list", f"key=layers config={origin}")
    cfg = NugopelConfig(vocab=k.integer("vocab"), width=k.integer("width"), eps=Keys(_object(obj, "norm", origin), origin).number("eps"))
    for i, entry in enumerate(layers):
        if not isinstance(entry, dict):
            raise AlofaError("parse", "a layer must be an object", f"layers[{i}] config={origin}")
        kind = Keys(entry, origin).string("type")
        cfg.layers.append(NugopelLayer(kind, _read_mixer(kind, _object(entry, "mixer", origin), origin), _read_mlp(entry.get("mlp"), origin)))
    cfg.validate(origin)
    return cfg


def to_json(cfg: NugopelConfig) -> dict:
    layers = []
    for layer in cfg.layers:
        m, f = layer.mixer, layer.mlp
        mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
        if layer.type == "latent_attention":
            mixer["kv_rank"] = m.kv_rank
            if m.kv_from is not None:
                mixer["kv_from"] = m.kv_from
        else:
            mixer.update({"kv_heads": m.kv_heads, "rot": {"base": m.rot_base, "dims": m.rot_dims}})
            if m.rot_scaling is not None:
                mixer["rot"]["scaling"] = dict(m.rot_scaling)
            if m.window is not None:
                mixer["mask"] = {"size": m.window}
        mlp = None
        if f is not None:
            mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            if f.shared_ff:
                mlp["shared"] = {"ff": f.shared_ff}
        layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
    return {"architecture": NAME, "vocab": cfg.vocab, "width": cfg.width, "norm": {"eps": cfg.eps}, "layers": layers}


def build_spec(cfg: NugopelConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.eps

    def norm(name: str, prefix: str = "") -> PartSpec:
        return PartSpec("rmsnorm", {"size": width, "eps": eps, "weight_name": name, "weight_offset": 1.0}, prefix=prefix)

    layers, run = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m, f = layer.mixer, layer.mlp
        if layer.type == "latent_attention":
            mixer = PartSpec("latent_attention", {"hidden_size": width, "heads": m.heads, "dim": m.dim, "rot_dim": 0, "vdim": m.vdim, "kv_rank": m.kv_rank, "q_rank": 0,
                                                  "scale": m.scale, "eps": eps, "sink": False, "window": None, "gate": "channel", "own_latent": m.kv_from is None}, prefix=p + "mix.")
            run.append(RunEntry(i, m.kv_from))
        else:
            rotary = PartSpec("rotary_interleaved", {"dims": m.rot_dims, "base": m.rot_base, "layout": "halves",
                                                     "scaling": {"kind": "wavelength", **m.rot_scaling} if m.rot_scaling is not None else None})
            mixer = PartSpec("normed_attention", {"hidden_size": width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                                                  "qk_norm": True, "norm_weight": True, "norm_over": "projection", "eps": eps, "position": rotary, "window": m.window,
                                                  "sink": SINK}, prefix=p + "mix.")
            run.append(RunEntry(i))
        block = {"mixer": mixer, "mixer_norm": norm("norm1", p), "mixer_post_norm": norm("norm1b", p), "feed_forward": None}
        if f is not None:
            block["feed_forward"] = PartSpec("routed_experts", {"hidden_size": width, "experts": f.experts, "top": f.top, "expert_ff": f.ff, "shared_ff": f.shared_ff,
                                                                "activation": "relu_squared", "score": "softmax", "renormalize": True}, prefix=p + "mlp.")
            block["feed_forward_norm"], block["feed_forward_post_norm"] = norm("norm2", p), norm("norm2b", p)
        layers.append(LayerSpec(PartSpec("sandwich_residual", block, prefix=p)))
    spec = ModelSpec(
        architecture=NAME, hidden_size=width, vocab_size=cfg.vocab, max_position=MAX_POSITION,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": width, "weight_name": "embed"}),
        layers=layers, run=run, final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": width, "tied_to": None, "weight_name": "head"}),
    )
    spec.validate()
    return spec


register_architecture(Architecture(NAME, read_config, build_spec, to_json), replace=True)
