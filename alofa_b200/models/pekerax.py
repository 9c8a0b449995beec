"""Pekerax: a pre-norm decoder (layer norms with weight and bias) whose layers,
listed one by one in config.json, have one of two mixers and optionally a
feed-forward:

* ``attention``: softmax attention without rotation.  q and k are each RMS
  normed over the whole projection with plain weights; a bias that grows with
  the distance of query and key (one slope per head) is taken off the scores;
  a sliding window beside which a request's first tokens stay visible; a
  learned sink per head in the softmax's denominator; values that (``v_mix``)
  are mixed with those of the first such layer; a sigmoid gate per head.
  Keys and values may have different head sizes;
* ``delta``: the gated delta rule with one decay per head, short convolutions
  on q, k and v, and a gated norm on the output.

The feed-forward is dense or a mixture of experts, both with the clamped gate
``g sigmoid(1.702 g) (u + 1)``; experts are chosen by softmax scores among the
best groups of neighbouring experts, a group's score being its largest.  The
embedding rows are multiplied by ``embedding.scale``; the head is the embedding
table without it.  This file only reads the architecture's config keys and
describes the model as a :class:`~alofa_b200.config.spec.ModelSpec`; the parts
it names live in :mod:`alofa_b200.parts` and know nothing about Pekerax.

config.json keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``,
``embedding.scale``, ``layers[i].type``, ``layers[i].mixer`` (attention:
``heads, kv_heads, dim, vdim, scale, v_mix, mask.{size, keep_first}``; delta:
``heads, kv_heads, dim, vdim, conv``) and ``layers[i].mlp`` (null, ``{kind:
dense, ff, limit}`` or ``{kind: moe, expert.{ff, limit}, router.{experts, top,
groups.{count, keep}}}``).  Absent ``mask``: every key; absent ``groups``: every
expert; absent ``limit``: no clamp.  Tensor names: ``embed``, ``l<i>.norm1``,
``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm`` (``.b`` for the
norms' biases)."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

from ..config.json_reader import Keys
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..errors import AlofaError

NAME = "Pekerax"
MAX_POSITION = 1 << 24  # distances are fp32 in the attention kernels: whole numbers are exact up to here
GATE_ALPHA = 1.702  # g * sigmoid(1.702 g) * (u + 1)
RENORM_EPS = 1e-20  # added to the sum the chosen experts' scores are divided by


@dataclass
class BiasedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    v_mix: bool = False
    window: Optional[int] = None
    keep_first: int = 0


@dataclass
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass
class FeedForwardConfig:
    kind: str  # "dense" or "moe"
    ff: int  # dense: the inner size; moe: one expert's
    limit: Optional[float] = None
    experts: int = 0
    top: int = 0
    groups: Optional[dict] = None  # count, keep


@dataclass
class PekeraxLayer:
    type: str
    mixer: object
    mlp: Optional[FeedForwardConfig]


@dataclass
class PekeraxConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float = 1.0
    layers: list = field(default_factory=list)

    def validate(self, origin: str = "") -> None:
        def need(ok, what, detail):
            if not ok:
                raise AlofaError("parse", what, f"{detail} config={origin}")

        need(self.vocab > 0 and self.width > 0, "vocab and width must be positive", f"vocab={self.vocab} width={self.width}")
        need(self.eps > 0, "norm.eps must be positive", f"eps={self.eps}")
        need(len(self.layers) > 0, "layers must not be empty", "layers=[]")
        mixed = set()
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            where = f"layers[{i}].mixer={m}"
            need(min(m.heads, m.kv_heads, m.dim, m.vdim) > 0 and m.heads % m.kv_heads == 0, "kv_heads must divide heads, sizes must be positive", where)
            if layer.type == "attention":
                need(m.window is None or m.window > 0, "mask.size must be positive", where)
                need(m.keep_first >= 0, "mask.keep_first must not be negative", where)
                if m.v_mix:
                    mixed.add(m.kv_heads * m.vdim)
            else:
                need(m.conv > 0, "conv must be positive", where)
            f = layer.mlp
            if f is not None:
                where = f"layers[{i}].mlp={f}"
                need(f.ff > 0, "the feed-forward's inner size must be positive", where)
                need(f.limit is None or f.limit > 0, "limit must be positive", where)
                if f.kind == "moe":
                    need(0 < f.top <= f.experts, "router.top must lie in [1, experts]", where)
                    g = f.groups
                    need(g is None or (g["count"] > 0 and f.experts % g["count"] == 0 and 0 < g["keep"] <= g["count"] and g["keep"] * (f.experts // g["count"]) >= f.top),
                         "router.groups: count must divide experts, and the groups kept must hold at least top experts", where)
        need(len(mixed) <= 1, "layers that mix their values must have the same number of them", f"kv_heads * vdim={sorted(mixed)}")


def _object(obj: dict, key: str, origin: str) -> dict:
    value = obj.get(key)
    if not isinstance(value, dict):
        raise AlofaError("parse", "config key must be an object", f"key={key} config={origin}")
    return value


def _read_mixer(kind: str, obj: dict, origin: str):
    k = Keys(obj, origin)
    if kind == "attention":
        window, keep = None, 0
        if isinstance(obj.get("mask"), dict):
            mk = Keys(obj["mask"], origin)
            window, keep = mk.integer("size"), mk.integer("keep_first", 0)
        return BiasedAttentionConfig(k.integer("heads"), k.integer("kv_heads"), k.integer("dim"), k.integer("vdim"), k.number("scale"), k.boolean("v_mix", False), window, keep)
    if kind == "delta":
        return DeltaConfig(k.integer("heads"), k.integer("kv_heads"), k.integer("dim"), k.integer("vdim"), k.integer("conv"))
    raise AlofaError("parse", "unknown layer type", f"type={kind} config={origin}")


def _limit(k: Keys) -> Optional[float]:
    return k.number("limit") if k.has("limit") else None


def _read_mlp(obj, origin: str) -> Optional[FeedForwardConfig]:
    if obj is None:
        return None
    if not isinstance(obj, dict):
        raise AlofaError("parse", "mlp must be an object or null", f"config={origin}")
    k = Keys(obj, origin)
    kind = k.string("kind")
    if kind == "dense":
        return FeedForwardConfig("dense", k.integer("ff"), _limit(k))
    if kind == "moe":
        ro = _object(obj, "router", origin)
        r, e = Keys(ro, origin), Keys(_object(obj, "expert", origin), origin)
        groups = None
        if isinstance(ro.get("groups"), dict):
            gk = Keys(ro["groups"], origin)
            groups = {"count": gk.integer("count"), "keep": gk.integer("keep")}
        return FeedForwardConfig("moe", e.integer("ff"), _limit(e), r.integer("experts"), r.integer("top"), groups)
    raise AlofaError("parse", "unknown mlp kind", f"kind={kind} config={origin}")


def read_config(obj: dict, origin: str) -> PekeraxConfig:
    k = Keys(obj, origin)
    layers = obj.get("layers")
    if not isinstance(layers, list):
        raise AlofaError("parse", "config key must be a list", f"key=layers config={origin}")
    cfg = PekeraxConfig(vocab=k.integer("vocab"), width=k.integer("width"), eps=Keys(_object(obj, "norm", origin), origin).number("eps"),
                        embedding_scale=Keys(_object(obj, "embedding", origin), origin).number("scale", 1.0) if obj.get("embedding") is not None else 1.0)
    for i, entry in enumerate(layers):
        if not isinstance(entry, dict):
            raise AlofaError("parse", "a layer must be an object", f"layers[{i}] config={origin}")
        kind = Keys(entry, origin).string("type")
        cfg.layers.append(PekeraxLayer(kind, _read_mixer(kind, _object(entry, "mixer", origin), origin), _read_mlp(entry.get("mlp"), origin)))
    cfg.validate(origin)
    return cfg


def to_json(cfg: PekeraxConfig) -> dict:
    def limited(entry: dict, limit) -> dict:
        return entry if limit is None else {**entry, "limit": limit}

    layers = []
    for layer in cfg.layers:
        m, f = layer.mixer, layer.mlp
        mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim}
        if layer.type == "attention":
            mixer.update({"scale": m.scale, "v_mix": m.v_mix})
            if m.window is not None:
                mixer["mask"] = {"size": m.window, "keep_first": m.keep_first}
        else:
            mixer["conv"] = m.conv
        if f is None:
            mlp = None
        elif f.kind == "dense":
            mlp = limited({"kind": "dense", "ff": f.ff}, f.limit)
        else:
            router = {"experts": f.experts, "top": f.top}
            if f.groups is not None:
                router["groups"] = dict(f.groups)
            mlp = {"kind": "moe", "expert": limited({"ff": f.ff}, f.limit), "router": router}
        layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
    return {"architecture": NAME, "vocab": cfg.vocab, "width": cfg.width, "norm": {"eps": cfg.eps}, "embedding": {"scale": cfg.embedding_scale}, "layers": layers}


def build_spec(cfg: PekeraxConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.eps

    def norm(name: str, prefix: str = "") -> PartSpec:
        return PartSpec("layernorm", {"size": width, "eps": eps, "weight_name": name}, prefix=prefix)

    layers = []
    mixed = False  # whether a layer before has left its values for the later ones to mix in
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m, f = layer.mixer, layer.mlp
        if layer.type == "attention":
            mix = None
            if m.v_mix:
                mix, mixed = ("later" if mixed else "first"), True
            mixer = PartSpec("normed_attention", {"hidden_size": width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                                                  "qk_norm": True, "norm_weight": True, "norm_over": "projection", "eps": eps, "distance_bias": True, "window": m.window,
                                                  "keep_first": m.keep_first, "sink": "learned", "value_mix": mix, "gate": True}, prefix=p + "mix.")
        else:
            mixer = PartSpec("gated_delta", {"hidden_size": width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv, "eps": eps,
                                             "decay_per": "head", "low_rank": False, "gate": "silu"}, prefix=p + "mix.")
        block = {"mixer": mixer, "mixer_norm": norm("norm1", p), "feed_forward": None}
        if f is not None:
            gate = {"gated": True, "activation": "clamped_silu", "gate_alpha": GATE_ALPHA, "gate_limit": f.limit}
            if f.kind == "dense":
                block["feed_forward"] = PartSpec("mlp", {"hidden_size": width, "intermediate_size": f.ff, **gate}, prefix=p + "mlp.")
            else:
                block["feed_forward"] = PartSpec("routed_experts", {"hidden_size": width, "experts": f.experts, "top": f.top, "expert_ff": f.ff, **gate, "score": "softmax",
                                                                    "renormalize": True, "renorm_eps": RENORM_EPS, "groups": f.groups["count"] if f.groups else 1,
                                                                    "keep": f.groups["keep"] if f.groups else 1, "group_score": "best"}, prefix=p + "mlp.")
            block["feed_forward_norm"] = norm("norm2", p)
        layers.append(LayerSpec(PartSpec("prenorm_residual", block, prefix=p)))
    spec = ModelSpec(
        architecture=NAME, hidden_size=width, vocab_size=cfg.vocab, max_position=MAX_POSITION,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": width, "weight_name": "embed", "scale": cfg.embedding_scale}),
        layers=layers, run=[RunEntry(i) for i in range(len(layers))], final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": width, "tied_to": "embed", "weight_name": "embed"}),
    )
    spec.validate()
    return spec


register_architecture(Architecture(NAME, read_config, build_spec, to_json), replace=True)
