"""Typed view of a Sevelorn ``config.json``.

The file lists its layers one by one: ``layers[i] = {"type", "mixer", "mlp"}``.  ``type`` names the mixer (``retention``,
``attention``; a numeric suffix, as in ``attention_2``, marks a further set of sizes of the same kind), ``mixer`` holds its
sizes and constants, ``mlp`` the feed-forward or null for a layer without one.

* ``retention``: ``heads``, ``dim``, ``vdim``, ``decay`` (one number per head), ``rot.dims``, ``rot.base``.
* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``.  ``kv_from: j``: the layer has no keys and values of
  its own and reads layer j's; layer j makes its own, and its kv heads and head sizes are this layer's.
* ``mlp.kind`` ``dense``: ``ff``.  ``moe``: ``router.experts``, ``router.top``, ``expert.ff``.

Top level: ``vocab``, ``width``, ``streams``, ``norm.eps``, ``canon.taps``, ``embedding.scale``.  Every size and constant is
read from the file; a missing key, a wrong type or an unknown kind is an error that names the key.  Parts that a file
leaves out (``rot``, ``streams``, ``canon``, ``embedding``) are switched off.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

from .fields import need as _need, positive as _positive
from .model_config import ConfigError

ARCHITECTURE = "Sevelorn"


@dataclass
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: list                       # one number per head
    rot_dims: int                     # 0: nothing is turned
    rot_base: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "RetentionConfig":
        heads = _positive(_need(d, "heads", int, where), where + ".heads")
        dim = _positive(_need(d, "dim", int, where), where + ".dim")
        vdim = _positive(_need(d, "vdim", int, where, default=dim, required=False), where + ".vdim")
        decay = d.get("decay")
        if (not isinstance(decay, list) or len(decay) != heads
                or any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay)):
            raise ConfigError(f"config.json: '{where}.decay' must be a list of one number per head ({heads})")
        dims, base = 0, 10000.0
        if d.get("rot") is not None:
            w = where + ".rot"
            dims = _need(d["rot"], "dims", int, w)
            if dims < 0 or dims % 2 or dims > dim:
                raise ConfigError(f"config.json: '{w}.dims' must be even, not negative and at most '{where}.dim'")
            base = _need(d["rot"], "base", float, w)
            if dims and (base <= 0 or base == 1.0):
                raise ConfigError(f"config.json: '{w}.base' must be positive and not 1")
        return cls(heads, dim, vdim, [float(x) for x in decay], dims, base)


@dataclass
class GatedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    kv_from: Optional[int]            # the layer whose keys and values this one reads (None: its own)

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "GatedAttentionConfig":
        heads = _positive(_need(d, "heads", int, where), where + ".heads")
        kv = _positive(_need(d, "kv_heads", int, where, default=heads, required=False), where + ".kv_heads")
        if heads % kv:
            raise ConfigError(f"config.json: '{where}.heads' must be a multiple of '{where}.kv_heads'")
        dim = _positive(_need(d, "dim", int, where), where + ".dim")
        vdim = _positive(_need(d, "vdim", int, where, default=dim, required=False), where + ".vdim")
        return cls(heads, kv, dim, vdim, _need(d, "scale", float, where), _need(d, "kv_from", int, where, required=False))


@dataclass
class MlpConfig:
    kind: str                         # "dense" | "moe"
    ff: int                           # dense: its width; moe: an expert's
    experts: int = 0
    top: int = 0

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "MlpConfig":
        kind = _need(d, "kind", str, where)
        if kind == "dense":
            return cls("dense", _positive(_need(d, "ff", int, where), where + ".ff"))
        if kind == "moe":
            r = _need(d, "router", dict, where)
            experts = _positive(_need(r, "experts", int, where + ".router"), where + ".router.experts")
            top = _positive(_need(r, "top", int, where + ".router"), where + ".router.top")
            if top > experts:
                raise ConfigError(f"config.json: '{where}.router.top' must be at most '{where}.router.experts'")
            ff = _positive(_need(_need(d, "expert", dict, where), "ff", int, where + ".expert"), where + ".expert.ff")
            return cls("moe", ff, experts, top)
        raise ConfigError(f"config.json: '{where}.kind' is {kind!r}; known: dense, moe")


MIXER_KINDS = {"retention": RetentionConfig, "attention": GatedAttentionConfig}


def _kind_of(name: str):
    head, sep, tail = name.rpartition("_")
    return head if sep and tail.isdigit() and head else name


@dataclass
class SevelornLayer:
    type: str
    mixer: object
    mlp: Optional[MlpConfig]


@dataclass
class SevelornConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    streams: int
    taps: int                         # of the convolution over a mixer's input; 0: there is none
    eps: float
    embed_scale: float
    layers: list = field(default_factory=list)
    raw: dict = field(default_factory=dict)
    eos_token_id: int = -1

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict) -> "SevelornConfig":
        layers_raw = d.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(layers_raw):
            where = f"layers[{i}]"
            typ = _need(L, "type", str, where)
            kind = MIXER_KINDS.get(_kind_of(typ))
            if kind is None:
                raise ConfigError(f"config.json: '{where}.type' is {typ!r}; known: {', '.join(sorted(MIXER_KINDS))} "
                                  "(with a numeric suffix for further sets of sizes)")
            mixer = kind.from_dict(_need(L, "mixer", dict, where), where + ".mixer")
            mlp = MlpConfig.from_dict(L["mlp"], where + ".mlp") if L.get("mlp") is not None else None
            layers.append(SevelornLayer(typ, mixer, mlp))
        for i, L in enumerate(layers):
            j = getattr(L.mixer, "kv_from", None)
            if j is None:
                continue
            where = f"layers[{i}].mixer.kv_from"
            if not (0 <= j < i) or not isinstance(layers[j].mixer, GatedAttentionConfig) or layers[j].mixer.kv_from is not None:
                raise ConfigError(f"config.json: '{where}' must name an earlier attention layer that makes its own keys and values")
            o, m = layers[j].mixer, L.mixer
            if (o.kv_heads, o.dim, o.vdim) != (m.kv_heads, m.dim, m.vdim):
                raise ConfigError(f"config.json: '{where}': layer {j}'s kv_heads, dim and vdim must equal this layer's")
        taps = 0
        if d.get("canon") is not None:
            taps = _positive(_need(d["canon"], "taps", int, "canon"), "canon.taps")
        scale = 1.0
        if d.get("embedding") is not None:
            scale = _need(d["embedding"], "scale", float, "embedding", default=1.0, required=False)
        eos = d.get("eos_token_id", -1)
        return cls(architecture=d.get("architecture", ARCHITECTURE),
                   vocab_size=_positive(_need(d, "vocab", int, ""), "vocab"),
                   hidden_size=_positive(_need(d, "width", int, ""), "width"),
                   streams=_positive(_need(d, "streams", int, "", default=1, required=False), "streams"), taps=taps,
                   eps=_need(_need(d, "norm", dict, ""), "eps", float, "norm"), embed_scale=scale, layers=layers,
                   raw=dict(d), eos_token_id=int(eos) if isinstance(eos, int) and not isinstance(eos, bool) else -1)

    def to_dict(self) -> dict:
        return dict(self.raw)
